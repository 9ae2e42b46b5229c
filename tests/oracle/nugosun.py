"""Plain, slow restatement of the Nugosun decoder for the tests: one function per mechanism, PyTorch
on the CPU in the precision of its inputs, no cache (every call sees a whole sequence), nothing
shared with the package. ``config`` is the checkpoint's config.json, ``weights`` maps its tensor
names to tensors."""
from __future__ import annotations

import math

import torch
from torch.nn.functional import silu, softplus

from .rodapel import heads_first, heads_last, rms_norm, rotate_pairs, softmax_attention, under, visible


def offset_norm(x, eps, w):
    """RMS norm whose weight is stored around zero."""
    return rms_norm(x, eps, 1.0 + w)


# ------------------------------------------------------------------ recurrences
def outer_recurrence(q, k, v, decay):
    """q, k, decay [heads, T, n], v [heads, T, d]: S = diag(decay) S + k v^T, then o = S^T q."""
    heads, t, n = q.shape
    s = torch.zeros(heads, n, v.shape[-1], dtype=q.dtype)
    out = []
    for i in range(t):
        s = decay[:, i, :, None] * s + k[:, i, :, None] * v[:, i, None, :]
        out.append((s * q[:, i, :, None]).sum(1))
    return torch.stack(out, 1)


def channel_decay(w, m, h):
    """sigmoid(z)^(1 / tau) per key channel, [heads, T, dim]."""
    z = (h @ w["a1"].T) @ w["a2"].T + w["a2.b"]
    return heads_first(torch.exp(torch.nn.functional.logsigmoid(z) / m["tau"]), m["heads"])


def gated_linear_attention(w, m, eps, h):
    hd = m["heads"]
    q, k, v = (heads_first(h @ w[s].T, hd) for s in "qkv")
    o = outer_recurrence(q * m["dim"] ** -0.5, k, v, channel_decay(w, m, h))
    return (heads_last(rms_norm(o, eps, w["norm"])) * silu(h @ w["g"].T)) @ w["o"].T


def causal_conv(x, taps, bias):
    """x [T, C], taps [C, n] (the last one multiplies the current token): depthwise, zeros before the start."""
    t, n = len(x), taps.shape[1]
    padded = torch.cat([torch.zeros(n - 1, x.shape[1], dtype=x.dtype), x])
    return sum(padded[j:j + t] * taps[:, j] for j in range(n)) + bias


def grouped_gated_norm(y, gate, groups, eps, w):
    """The gate first, then every one of the equal groups over its own root mean square."""
    y = y * silu(gate)
    return rms_norm(y.reshape(len(y), groups, -1), eps).reshape(len(y), -1) * w


def state_space(w, m, eps, h):
    hd, vd, n, g = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = hd * vd
    z, xbc, dt = torch.split(h @ w["in"].T, [inner, inner + 2 * g * n, hd], dim=-1)
    x, b, c = torch.split(silu(causal_conv(xbc, w["conv"], w["conv.b"])), [inner, g * n, g * n], dim=-1)
    dt = softplus(dt + w["dt_bias"])                                         # [T, heads]
    b, c = (heads_first(s, g).repeat_interleave(hd // g, 0) for s in (b, c))   # [heads, T, n]
    x = heads_first(x, hd)
    decay = torch.exp(-torch.exp(w["A_log"]) * dt).T[:, :, None].expand(-1, -1, n)
    y = outer_recurrence(c, b * dt.T[:, :, None], x, decay) + w["D"][:, None, None] * x
    return grouped_gated_norm(heads_last(y), z, m["norm_groups"], eps, w["norm"]) @ w["o"].T


# ------------------------------------------------------------------ attention
def turn_frequencies(rot):
    """(angle per position of every pair, factor of cos and sin)."""
    dims, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    s = rot.get("scaling")
    if not s:
        return f, 1.0
    where = lambda turns: dims * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))   # noqa: E731
    lo, hi = max(math.floor(where(s["fast"])), 0), min(math.ceil(where(s["slow"])), dims - 1)
    ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(dims // 2)]
    return [a / s["factor"] * r + a * (1 - r) for a, r in zip(f, ramp)], 0.1 * math.log(s["factor"]) + 1.0


def rotate_halves(x, rot):
    """x [heads, T, d]: value i of the first ``dims`` turns with value i + dims / 2."""
    f, grow = turn_frequencies(rot)
    half = len(f)
    a = torch.arange(x.shape[1], dtype=torch.float64)[:, None] * torch.tensor(f, dtype=torch.float64)
    cos, sin = (torch.cos(a) * grow).to(x.dtype), (torch.sin(a) * grow).to(x.dtype)
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., 2 * half:]], -1)


def same_chunk(t, size):
    i = torch.arange(t) // size
    return visible(t) & (i[:, None] == i[None, :])


def chunked_attention(w, m, eps, h):
    hd, kv = m["heads"], m["kv_heads"]
    proj = lambda s, n: heads_first(h @ w[s].T + w[s + ".b"], n)              # noqa: E731
    q, k = (rms_norm(rotate_halves(proj(s, n), m["rot"]), eps) for s, n in (("q", hd), ("k", kv)))
    k, v = (s.repeat_interleave(hd // kv, 0) for s in (k, proj("v", kv)))
    s = q @ k.transpose(1, 2) * m["scale"]
    if m.get("softcap"):
        s = m["softcap"] * torch.tanh(s / m["softcap"])
    seen = same_chunk(len(h), m["mask"]["size"]) if m.get("mask") else visible(len(h))
    return heads_last(softmax_attention(s, seen, v)) @ w["o"].T


def side_by_side(w, m, eps, h):
    left = chunked_attention(under(w, "left."), m["left"], eps, h)
    right = state_space(under(w, "right."), m["right"], eps, h)
    return m["left_scale"] * left + m["right_scale"] * right


def latent_rows(w, m, eps, h):
    """(normed latent [T, rank], rotated key part [T, rot])."""
    down, rank = h @ w["dkv"].T, m["kv_rank"]
    return rms_norm(down[:, :rank], eps, w["dkv.norm"]), rotate_pairs(down[:, rank:], m["rot"]["base"], m["rot"]["dims"])


def latent_attention(w, m, eps, h, rows):
    """``rows``: what ``latent_rows`` gave, of this layer or of the one it shares with."""
    hd, dim = m["heads"], m["dim"]
    c, kr = rows
    q = heads_first(rms_norm(h @ w["dq"].T, eps, w["dq.norm"]) @ w["uq"].T, hd)
    qn, qr = q[..., :dim], rotate_pairs(q[..., dim:], m["rot"]["base"], m["rot"]["dims"])
    k, v = heads_first(c @ w["uk"].T, hd), heads_first(c @ w["uv"].T, hd)
    s = (qn @ k.transpose(1, 2) + qr @ kr.T) * m["scale"]
    return heads_last(softmax_attention(s, visible(len(h)), v)) @ w["o"].T


# ------------------------------------------------------------------ feed-forward
def swiglu(gate, up, down, h):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def route(router, bias, top, h):
    """(experts [T, top], weights [T, top]): the largest logits, weighted by the softmax over them alone."""
    z, idx = torch.topk(h @ router.T + bias, top, dim=-1)
    return idx, torch.softmax(z, dim=-1)


def expert_mix(w, mlp, h):
    idx, wt = route(w["router"], w["router.b"], mlp["router"]["top"], h)
    y = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        t, s = (idx == e).nonzero(as_tuple=True)
        if len(t):
            y[t] += wt[t, s, None] * swiglu(w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], h[t])
    return y


def feed_forward(w, mlp, h):
    return expert_mix(w, mlp, h) if mlp["kind"] == "moe" else swiglu(w["gate"], w["up"], w["down"], h)


def forward(config, weights, tokens, observe=None):
    """Logits [T, vocab] of one whole sequence. ``observe(layer, residual)`` after every layer."""
    eps = config["norm"]["eps"]
    x = weights["embed"][torch.as_tensor(tokens, dtype=torch.long)] * config["embedding"]["scale"]
    shared = {}
    for i, layer in enumerate(config["layers"]):
        w, m = under(weights, f"l{i}."), layer["mixer"]
        mix, h = under(w, "mix."), offset_norm(x, eps, w["norm1"])
        if layer["type"] == "latent_attention":
            src = m.get("kv_from", i)
            if src == i:
                shared[i] = latent_rows(mix, m, eps, h)
            y = latent_attention(mix, m, eps, h, shared[src])
        else:
            y = {"gla": gated_linear_attention, "parallel": side_by_side}[layer["type"]](mix, m, eps, h)
        if layer.get("mlp"):
            y = y + feed_forward(under(w, "mlp."), layer["mlp"], offset_norm(x, eps, w["norm2"]))
        x = x + y
        if observe is not None:
            observe(i, x)
    return offset_norm(x, eps, weights["final.norm"]) @ weights["embed"].T
