"""Plain, slow restatement of the Nizorax decoder for the tests: one function per mechanism, PyTorch on the CPU in the
precision of its inputs, no cache (every call sees a whole sequence), nothing shared with the package. ``config`` is the
checkpoint's config.json, ``weights`` maps its tensor names to tensors."""
from __future__ import annotations

import math

import torch

from .nugosun import swiglu
from .rodapel import heads_first, heads_last, rms_norm, softmax_attention, under, visible


def layer_norm(x, eps, w, b):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def short_conv(h, taps):
    """h [T, width] plus its causal depthwise convolution; taps [width, n], the last one multiplies the current token."""
    n = taps.shape[1]
    past = torch.cat([h.new_zeros(n - 1, h.shape[1]), h])
    return h + sum(past[j:j + len(h)] * taps[:, j] for j in range(n))


def runs(config):
    """The layers in the order in which they run."""
    order, loop = list(range(len(config["layers"]))), config.get("loop")
    if not loop:
        return order
    a, b = loop["start"], loop["stop"]
    return order[:a] + order[a:b] * loop["times"] + order[b:]


# ------------------------------------------------------------------ mixers
def silu(z):
    return z / (1 + torch.exp(-z))


def decayed_state(q, k, v, decay):
    """q, k [heads, T, n], v [heads, T, d], one decay per head: S = decay S + k v^T, then o = S^T q."""
    s = q.new_zeros(q.shape[0], q.shape[2], v.shape[2])
    out = []
    for t in range(q.shape[1]):
        s = decay[:, None, None] * s + torch.einsum("hn,hd->hnd", k[:, t], v[:, t])
        out.append(torch.einsum("hnd,hn->hd", s, q[:, t]))
    return torch.stack(out, 1)


def lightning(w, m, eps, h):
    q, k, v = (heads_first(silu(h @ w[n].T), m["heads"]) for n in "qkv")
    o = heads_last(decayed_state(q, k, v, torch.tensor(m["decay"], dtype=h.dtype)))
    return (rms_norm(o, eps, w["norm"]) * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def turn_frequencies(rot):
    """Angle per position of every pair."""
    f = [rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)]
    s = rot.get("scaling")
    if not s:
        return f
    out = []
    for a in f:
        turns = s["original"] * a / (2 * math.pi)              # over the original length
        if turns > s["high"]:
            out.append(a)
        elif turns < s["low"]:
            out.append(a / s["factor"])
        else:
            mix = (turns - s["low"]) / (s["high"] - s["low"])
            out.append((1 - mix) * a / s["factor"] + mix * a)
    return out


def rotate_neighbours(x, rot):
    """x [..., T, d]: values 2i and 2i + 1 of the first ``dims`` turn together."""
    dims = rot["dims"]
    a = torch.arange(x.shape[-2], dtype=torch.float64)[:, None] * torch.tensor(turn_frequencies(rot), dtype=torch.float64)
    cos, sin = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    return torch.cat([torch.stack([u * cos - v * sin, v * cos + u * sin], -1).flatten(-2), x[..., dims:]], -1)


def map_weight(w, diff):
    """What the second map is multiplied by."""
    return torch.exp((w["lq1"] * w["lk1"]).sum()) - torch.exp((w["lq2"] * w["lk2"]).sum()) + diff


def two_maps(q, k, v, seen, scale, lam, diff, eps):
    """q [heads, 2, T, dim], k [groups, 2, T, dim], v [groups, T, vdim] -> [heads, T, vdim]: the maps' difference, normed."""
    per = q.shape[0] // k.shape[0]
    k, v = k.repeat_interleave(per, 0), v.repeat_interleave(per, 0)
    a = [softmax_attention(q[:, i] @ k[:, i].transpose(1, 2) * scale, seen, v) for i in (0, 1)]
    return rms_norm(a[0] - lam * a[1], eps) * (1 - diff)


def differential_attention(w, m, eps, h):
    hd, kv, t = m["heads"], m["kv_heads"], len(h)
    q, k = (rotate_neighbours(heads_first(h @ w[n].T, 2 * c), m["rot"]).reshape(c, 2, t, m["dim"])
            for n, c in (("q", hd), ("k", kv)))
    o = two_maps(q, k, heads_first(h @ w["v"].T, kv), visible(t, (m.get("mask") or {}).get("size")), m["scale"],
                 map_weight(w, m["diff"]), m["diff"], eps)
    return heads_last(o) @ w["o"].T


# ------------------------------------------------------------------ feed-forward
def poly_norm(z, eps, act):
    a, b, c, e = act
    return a * rms_norm(z, eps) + b * rms_norm(z ** 2, eps) + c * rms_norm(z ** 3, eps) + e


def route(router, r, h):
    """(experts [T, top], weights [T, top]): sigmoid scores; only experts of the best groups, by their two best."""
    s = torch.sigmoid(h @ router.T)
    g = r.get("groups")
    open_to = s
    if g:
        per = s.reshape(len(s), g["count"], -1)
        best = per.sort(-1, descending=True).values[..., :2].sum(-1)
        kept = torch.zeros_like(best, dtype=torch.bool).scatter(1, best.topk(g["keep"], -1).indices, True)
        open_to = torch.where(kept[..., None].expand_as(per).reshape_as(s), s, torch.full_like(s, -1.0))
    idx = open_to.topk(r["top"], -1).indices
    return idx, s.gather(1, idx) * r["scale"]


def expert_mix(w, mlp, h):
    idx, wt = route(w["router"], mlp["router"], h)
    y = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        t, s = (idx == e).nonzero(as_tuple=True)
        if len(t):
            y[t] += wt[t, s, None] * swiglu(w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], h[t])
    if mlp.get("shared"):
        y = y + swiglu(w["shared.gate"], w["shared.up"], w["shared.down"], h)
    return y


def feed_forward(w, mlp, eps, h):
    return expert_mix(w, mlp, h) if mlp["kind"] == "moe" else poly_norm(h @ w["up"].T, eps, w["act"]) @ w["down"].T


def forward(config, weights, tokens, observe=None):
    """Logits [T, vocab] of one whole sequence. ``observe(run, residual)`` after every layer run."""
    eps = config["norm"]["eps"]
    x = weights["embed"][torch.as_tensor(tokens, dtype=torch.long)] * config["embedding"]["scale"]
    for n, i in enumerate(runs(config)):
        layer, w = config["layers"][i], under(weights, f"l{i}.")
        norm = lambda v, name: layer_norm(v, eps, w[name], w[name + ".b"])      # noqa: E731
        mixer = {"lightning": lightning, "attention": differential_attention}[layer["type"]]
        h = short_conv(norm(x, "norm1"), w["canon1"])
        x = x + norm(mixer(under(w, "mix."), layer["mixer"], eps, h), "norm1b")
        if layer.get("mlp"):
            h = short_conv(norm(x, "norm2"), w["canon2"])
            x = x + norm(feed_forward(under(w, "mlp."), layer["mlp"], eps, h), "norm2b")
        if observe is not None:
            observe(n, x)
    h = layer_norm(x, eps, weights["final.norm"], weights["final.norm.b"])
    return h @ weights["head"].T * config["logit_scale"]
