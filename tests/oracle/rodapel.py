"""Plain, slow restatement of the Rodapel decoder for the tests: one function per mechanism, PyTorch
on the CPU in the precision of its inputs, no cache (every call sees a whole sequence), nothing
shared with the package. ``config`` is the checkpoint's config.json, ``weights`` maps its tensor
names to tensors."""
from __future__ import annotations

import math

import torch


def rms_norm(x, eps, weight=None):
    """Each row over its own root mean square, times the weight if there is one."""
    y = x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def heads_first(rows, heads):
    """[T, heads * d] -> [heads, T, d]."""
    t, n = rows.shape
    return rows.reshape(t, heads, n // heads).permute(1, 0, 2)


def heads_last(x):
    """[heads, T, d] -> [T, heads * d]."""
    return x.permute(1, 0, 2).reshape(x.shape[1], -1)


def visible(t, window=None):
    """[T, T]: may query i see key j. ``window``: only the last so many tokens, itself included."""
    i, j = torch.arange(t)[:, None], torch.arange(t)[None, :]
    m = j <= i
    return m if window is None else m & (i - j < window)


def softmax_attention(scores, mask, v):
    """scores [heads, T, T], v [heads, T, d]."""
    return torch.softmax(scores.masked_fill(~mask, -math.inf), dim=-1) @ v


def rotate_pairs(x, base, dims):
    """x [..., T, d]: neighbours (2i, 2i + 1) of the first ``dims`` values turned by position * base^(-2i / dims)."""
    t, i = x.shape[-2], torch.arange(dims // 2, dtype=torch.float64)
    a = torch.arange(t, dtype=torch.float64)[:, None] * base ** (-2.0 * i / dims)
    cos, sin = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * cos - v * sin
    out[..., 1:dims:2] = v * cos + u * sin
    return out


def window_attention(w, m, eps, h):
    """Grouped-query attention over a sliding window, per-head query / key norm, no positions, each
    head's output scaled by a sigmoid gate."""
    q = rms_norm(heads_first(h @ w["q"].T, m["heads"]), eps, w["q.norm"])
    k = rms_norm(heads_first(h @ w["k"].T, m["kv_heads"]), eps, w["k.norm"])
    v = heads_first(h @ w["v"].T, m["kv_heads"])
    group = m["heads"] // m["kv_heads"]
    k, v = k.repeat_interleave(group, 0), v.repeat_interleave(group, 0)
    o = softmax_attention(q @ k.transpose(1, 2) * m["scale"], visible(len(h), (m.get("mask") or {}).get("size")), v)
    gate = torch.sigmoid(h @ w["g"].T)                       # [T, heads]
    return heads_last(o * gate.T[:, :, None]) @ w["o"].T


def latent_attention(w, m, eps, h):
    """Keys and values expanded from one normed latent per token; one rotated key part for all heads."""
    hd, dim, rot, rank = m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    base, dims = m["rot"]["base"], m["rot"]["dims"]
    q = heads_first(h @ w["q"].T, hd)
    down = h @ w["dkv"].T
    c, kr = rms_norm(down[:, :rank], eps, w["dkv.norm"]), rotate_pairs(down[:, rank:], base, dims)
    qn, qr = q[..., :dim], rotate_pairs(q[..., dim:], base, dims)
    assert qr.shape[-1] == rot
    k, v = heads_first(c @ w["uk"].T, hd), heads_first(c @ w["uv"].T, hd)
    s = (qn @ k.transpose(1, 2) + qr @ kr.T) * m["scale"]
    return heads_last(softmax_attention(s, visible(len(h)), v)) @ w["o"].T


def token_shift(h, mu):
    """h + (the previous token's h - h) * mu, zeros before the first token."""
    prev = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (prev - h) * mu


def wkv_recurrence(r, k, v, decay, u):
    """All [heads, T, d] (u [heads, d]): o_t = (S + diag(u) k v^T)^T r, then S = diag(decay) S + k v^T."""
    heads, t, d = r.shape
    s = torch.zeros(heads, d, d, dtype=r.dtype)
    out = []
    for i in range(t):
        kv = k[:, i, :, None] * v[:, i, None, :]
        out.append(((s + u[:, :, None] * kv) * r[:, i, :, None]).sum(1))
        s = decay[:, i, :, None] * s + kv
    return torch.stack(out, 1)


def time_mix(w, m, eps, h):
    mix = {s: token_shift(h, w["mu." + s]) for s in "rkvgw"}
    r, k, v = (heads_first(mix[s] @ w[s].T, m["heads"]) for s in "rkv")
    gate = torch.nn.functional.silu(mix["g"] @ w["g"].T)
    decay = torch.exp(-torch.exp(torch.tanh(mix["w"] @ w["w1"].T) @ w["w2"].T + w["w0"]))
    o = wkv_recurrence(r, k, v, heads_first(decay, m["heads"]), w["u"])
    return (heads_last(rms_norm(o, eps)) * w["norm"] * gate) @ w["o"].T


def clamped_gate_ffn(gate, up, down, limit, h):
    g = (h @ gate.T).clamp(max=limit)
    u = (h @ up.T).clamp(min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ down.T


def route(router, correction, top, h):
    """(experts [T, top], weights [T, top]): chosen by softmax + correction, weighted by the softmax."""
    s = torch.softmax(h @ router.T, dim=-1)
    idx = torch.topk(s + correction, top, dim=-1).indices
    return idx, s.gather(1, idx)


def expert_mix(w, mlp, h):
    r, limit = mlp["router"], mlp["expert"]["limit"]
    idx, wt = route(w["router"], w["correction"], r["top"], h)
    y = torch.zeros_like(h)
    for t in range(len(h)):
        for e, a in zip(idx[t].tolist(), wt[t]):
            x = h[t:t + 1]
            if e < r["experts"]:
                x = clamped_gate_ffn(w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], limit, x)
            y[t] += a * x[0]
    return y


def feed_forward(w, mlp, h):
    if mlp["kind"] == "moe":
        return expert_mix(w, mlp, h)
    return clamped_gate_ffn(w["gate"], w["up"], w["down"], mlp["limit"], h)


MIXERS = {"attention": window_attention, "latent_attention": latent_attention, "wkv": time_mix}


def under(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(config, weights, tokens, observe=None):
    """Logits [T, vocab] of one whole sequence. ``observe(layer, residual)`` after every layer."""
    eps = config["norm"]["eps"]
    x = rms_norm(weights["embed"][torch.as_tensor(tokens, dtype=torch.long)], eps, weights["embed.norm"])
    for i, layer in enumerate(config["layers"]):
        w = under(weights, f"l{i}.")
        x = x + rms_norm(MIXERS[layer["type"]](under(w, "mix."), layer["mixer"], eps, x), eps, w["norm1"])
        if layer.get("mlp"):
            x = x + rms_norm(feed_forward(under(w, "mlp."), layer["mlp"], x), eps, w["norm2"])
        if observe is not None:
            observe(i, x)
    return rms_norm(x, eps, weights["final.norm"]) @ weights["head"].T
