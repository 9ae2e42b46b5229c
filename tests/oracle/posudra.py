"""Plain, slow restatement of the Posudra decoder for the tests: one function per mechanism, PyTorch
on the CPU in the precision of its inputs, no cache (every call sees a whole sequence), nothing
shared with the package. ``weights`` maps the checkpoint's tensor names to tensors."""
from __future__ import annotations

import math

import torch


def rms_norm(x, weight, eps):
    """Each row over its own root mean square, times the weight."""
    rms = torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)
    return x / rms * weight


def embed(table, tokens, scale):
    return table[torch.as_tensor(tokens, dtype=torch.long)] * scale


def split_heads(rows, heads):
    """[T, heads * d] -> [heads, T, d]."""
    t, n = rows.shape
    return rows.reshape(t, heads, n // heads).permute(1, 0, 2)


def soft_cap(score, cap):
    return cap * torch.tanh(score / cap)


def distance_bias(t, r1, r2, dtype):
    """[heads, T, T]: what is taken off the score of query i and key j <= i, per head."""
    pos = torch.arange(t, dtype=dtype)
    gap = (pos[:, None] - pos[None, :]).clamp(min=0)
    return r1[:, None, None] * torch.log(1 + r2[:, None, None] * gap)


def sink_softmax(scores, sink):
    """Softmax over the last dimension whose denominator also counts one entry of logit ``sink``
    (per head) that has no value. scores [heads, T, T] with -inf where a key is not visible."""
    top = torch.maximum(scores.amax(-1, keepdim=True), sink[:, None, None])
    e = torch.exp(scores - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink[:, None, None] - top))


def scored_attention(q, k, v, scale, temp, cap, r1, r2, sink):
    """q [heads, T, d], k and v per query head; causal over one sequence. Returns [heads, T, dv]."""
    t = q.shape[1]
    score = (q @ k.transpose(1, 2)) * scale
    score = score * temp[:, None, None]
    score = soft_cap(score, cap)
    score = score - distance_bias(t, r1, r2, q.dtype)
    visible = torch.ones(t, t, dtype=torch.bool).tril()
    score = score.masked_fill(~visible, -math.inf)
    return sink_softmax(score, sink) @ v


def repeat_groups(kv, heads):
    """Query head i uses key / value head i // (heads / groups)."""
    per = heads // kv.shape[0]
    return torch.stack([kv[i // per] for i in range(heads)])


def attention(h, w, mixer, eps):
    """h [T, width]; w maps 'q', 'k', ... to the layer's tensors. Returns [T, width]."""
    t, heads, groups = h.shape[0], mixer["heads"], mixer["kv_heads"]
    q = split_heads(rms_norm(h @ w["q"].T, w["q.norm"], eps), heads)
    k = split_heads(rms_norm(h @ w["k"].T, w["k.norm"], eps), groups)
    v = split_heads(h @ w["v"].T, groups)
    out = scored_attention(q, repeat_groups(k, heads), repeat_groups(v, heads), mixer["scale"], w["temp"],
                           mixer["softcap"], w["r1"], w["r2"], w["sink"])
    return out.permute(1, 0, 2).reshape(t, -1) @ w["o"].T


def xielu(z, p, q):
    """softplus(p) z^2 + z / 2 above zero, (1/2 + softplus(q)) (e^z - 1 - z) + z / 2 below."""
    ap, an = torch.nn.functional.softplus(p), 0.5 + torch.nn.functional.softplus(q)
    neg = torch.clamp(z, max=0)
    return torch.where(z > 0, ap * z * z + z / 2, an * (torch.expm1(neg) - neg) + z / 2)


def feed_forward(h, w):
    return xielu(h @ w["up"].T, w["act"][0], w["act"][1]) @ w["down"].T


def sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def layer(x, weights, index, entry, eps):
    """One parallel block: a single norm, both sublayers read it, each has its own layer scale."""
    w = sub(weights, f"l{index}.")
    h = rms_norm(x, w["norm1"], eps)
    delta = attention(h, sub(w, "mix."), entry["mixer"], eps) * w["ls1"]
    if entry.get("mlp") is not None:
        delta = delta + feed_forward(h, sub(w, "mlp.")) * w["ls2"]
    return x + delta


def forward(config, weights, tokens, dtype=torch.float64, want_layers=False):
    """Logits [T, vocab] of one sequence (and the residual stream after every layer)."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = embed(w["embed"], tokens, config["embedding"]["scale"])
    stream = []
    for i, entry in enumerate(config["layers"]):
        x = layer(x, w, i, entry, eps)
        stream.append(x)
    logits = rms_norm(x, w["final.norm"], eps) @ w["head"].T
    return (logits, torch.stack(stream)) if want_layers else logits
