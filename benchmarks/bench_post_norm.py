#!/usr/bin/env python
"""Prefill and decode throughput of the post-norm decoder (Rodapel) beside the framework's mixture-of-experts
transformer at equal size, and its kernels beside the like kernels of the framework's other models, each
against its roofline. Random weights, one GPU, bf16.

    python benchmarks/bench_post_norm.py [--sizes 2048,4096] [--layers 8] [--kernels]
    python bench.py --suite post_norm ...       # the same

Layers come in fours: windowed attention + dense, WKV + routed, latent attention + routed, windowed attention +
routed. Equal size: the transformer has the same width, heads (size 128), expert count and widths, top k, and
as many dense layers; its attention is full. Prefill: one prompt of ``--tokens``; decode: B sequences of
``--ctx`` cached tokens, one captured step per token. Timing: CUDA events after warm-up; the layers' weights
together exceed L2. Kernel times: graph-captured loops over all layers of a kind (each with its own weights
and pages), after a pause in which the clocks recover from the power cap. "roofline" is the largest of bytes /
copy bandwidth, tensor FLOPs / burst GEMM rate (MEASURED_PEAKS.json) and, for the recurrence, fp32 operations /
(SMs x 128 a clock at the top clock)."""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
from bench_parallel_block import VOCAB, ev_ms, graph_us, peaks  # noqa: E402

from rmlx_b200._lib import NativeError  # noqa: E402
from rmlx_b200.config import (ClampedFfSpec, FeedForwardType, LatentAttentionSpec, MoeConfig, PostNormLayerSpec,  # noqa: E402
                              RodapelConfig, RoutedFfSpec, TransformerConfig, WindowAttentionSpec, WkvSpec)
from rmlx_b200.models.rodapel import (Buffers, DenseFfWeights, LatentWeights, RodapelModel, RoutedFfWeights,  # noqa: E402
                                      StepContext, WindowWeights, WkvWeights, build_weights, random_tensors)
from rmlx_b200.models.ragged import Entry, RaggedBatch  # noqa: E402
from rmlx_b200.models.transformer import TransformerModel  # noqa: E402
from rmlx_b200.models.weights import random_on_device  # noqa: E402
from rmlx_b200.ops import decode as D  # noqa: E402
from rmlx_b200.ops import latent as L  # noqa: E402
from rmlx_b200.ops import parallel_block as P  # noqa: E402
from rmlx_b200.ops import post_norm as N  # noqa: E402
from rmlx_b200.ops import routed as R  # noqa: E402
from rmlx_b200.ops import wkv as W  # noqa: E402
from rmlx_b200.ops.gemm import GemmStatus, gemm_bf16  # noqa: E402
from rmlx_b200.ops.quantized import xgemm  # noqa: E402

HD, WINDOW, EXPERTS, IDENTITY, TOP = 128, 1024, 32, 8, 4
# width: (query heads, kv heads, dense inner width, expert inner width)
SIZES = {2048: (16, 4, 8192, 2048), 4096: (32, 8, 14336, 3584)}
FP32_OPS = 148 * 128 * 1.965e9


def rodapel_cfg(width: int, layers: int) -> RodapelConfig:
    hq, hkv, inner, ex = SIZES[width]
    win = WindowAttentionSpec(hq, hkv, HD, HD, HD ** -0.5, WINDOW)
    lat = LatentAttentionSpec(hq, 128, 64, 128, 512, 192 ** -0.5)
    moe = RoutedFfSpec(EXPERTS, IDENTITY, TOP, ex, 7.0)
    four = [PostNormLayerSpec(win, ClampedFfSpec(inner, 7.0)), PostNormLayerSpec(WkvSpec(width // 64, 64, 64), moe),
            PostNormLayerSpec(lat, moe), PostNormLayerSpec(win, moe)]
    return RodapelConfig(VOCAB, width, four * (layers // 4), 1e-6).validate()


def moe_cfg(width: int, layers: int, max_len: int) -> TransformerConfig:
    hq, hkv, inner, ex = SIZES[width]
    return TransformerConfig(hidden_size=width, num_heads=hq, num_kv_heads=hkv, head_dim=HD, num_layers=layers,
                             vocab_size=VOCAB, max_seq_len=max_len, ff_type=FeedForwardType.moe_(
                                 MoeConfig(EXPERTS, TOP, width, ex)), first_dense_layers=layers // 4,
                             dense_intermediate_dim=inner, name="moe").validate()


def filled_cache(model, batch: int, ctx: int, extra: int):
    bps = (ctx + extra + 15) // 16
    cache = model.new_cache(1 + batch * bps, max_seqs=batch, max_blocks_per_seq=bps)
    for s in range(batch):
        cache.add_sequence(s)
        cache.reserve(s, ctx)
        cache.commit(s, ctx)
    for pool in {id(p): p for p in cache.k + cache.v if p is not None}.values():
        pool.normal_(0, 1)
    return cache


def run_models(model, tokens, batches, ctx, steps=32):
    """tokens/s of a prompt and of decode at each batch size."""
    out = {}
    for t in tokens:
        ids = torch.randint(0, VOCAB, (t,), device=model.device)
        cache = model.new_cache(t // 16 + 2, max_seqs=1, max_blocks_per_seq=t // 16 + 1)

        def prompt():
            cache.add_sequence(0)
            model.prefill(ids, cache, 0)
            cache.free_sequence(0)

        out[f"prefill_{t}"] = round(t * 1e3 / ev_ms(prompt, 5), 1)
        del cache
    for b in batches:
        cache = filled_cache(model, b, ctx, 2 * steps + 32)
        eng = model.make_decode_engine(cache, b)
        eng.bind(list(range(b)), [1] * b)
        eng.reserve(2 * steps + 16)
        try:
            out[f"decode_b{b}"] = round(b * 1e3 / ev_ms(eng.step, steps, warmup=4), 1)
        except NativeError:              # a mat-vec that cannot stage this many rows of this width
            out[f"decode_b{b}"] = None
        del eng, cache
        torch.cuda.empty_cache()
    GemmStatus.check(model.device)
    return out


class Table:
    """One row per kernel: time, roofline and fraction, beside the like kernel of another model."""

    def __init__(self, width):
        self.width, (self.bw, self.fl) = width, peaks()

    def _frac(self, us, nbytes, flops, ops):
        floor = max(nbytes / self.bw, flops / self.fl, ops / FP32_OPS) * 1e6
        return round(us, 2), round(floor / us, 3)

    def add(self, phase, kernel, fns, cost, like=None, like_fns=None, like_cost=None):
        """``fns``: one callable per layer of the loop; costs: (bytes, tensor FLOPs[, fp32 operations])."""
        def timed(f, c):
            return self._frac(graph_us(lambda: [g() for g in f], len(f)), *c, *([0] * (3 - len(c))))
        us, frac = timed(fns, cost)
        row = {"width": self.width, "phase": phase, "kernel": kernel, "us": us, "of_roofline": frac}
        if like is not None:
            lus, lfrac = timed(like_fns, like_cost or cost)
            row.update({"like": like, "like_us": lus, "like_of_roofline": lfrac, "x": round(lfrac / frac, 2)})
        print(json.dumps(row), flush=True)


def kinds(model):
    ls = list(enumerate(model.w.layers))
    pick = lambda cls, part: [(i, getattr(l, part), l) for i, l in ls if isinstance(getattr(l, part), cls)]   # noqa: E731
    return (pick(WindowWeights, "mix"), pick(LatentWeights, "mix"), pick(WkvWeights, "mix"), pick(DenseFfWeights, "mlp"),
            pick(RoutedFfWeights, "mlp"))


def prefill_kernels(tab: Table, model: RodapelModel, t: int):
    from rmlx_b200.ops.attention import flash_prefill_paged
    cfg, d, dev, bf = model.cfg, model.cfg.width, model.device, torch.bfloat16
    win, lat, wkv, dense, moe = kinds(model)
    cache = model.new_cache(t // 16 + 2, max_seqs=1, max_blocks_per_seq=t // 16 + 1)
    cache.add_sequence(0)
    batch = RaggedBatch.plan([Entry(0, [1] * t)], cache, min(l.mixer.heads for l in cfg.layers), model._absorb)
    cache.reserve(0, t)
    batch.upload(dev)
    bufs = Buffers(t, dev)
    c = StepContext(t, bufs, cache, cache.block_table, batch.positions, batch.token_seq, batch.token_seq, batch.runs, batch)
    for pool in {id(p): p for p in cache.k + cache.v if p is not None}.values():
        pool.normal_()
    x, h = torch.randn(t, d, device=dev), torch.randn(t, d, dtype=bf, device=dev)
    y, res = torch.randn(t, d, device=dev), torch.randn(t, d, dtype=bf, device=dev)
    ph, row = f"prefill {t}", cache.block_table[0]
    gemm = lambda n, k, out=2: (n * k * 2 + t * (k * 2 + n * out), 2.0 * t * n * k)          # noqa: E731
    # windowed attention
    m = win[0][1].spec
    nq, nkv = m.heads * m.dim, m.kv_heads * m.dim
    raw = torch.randn(t, win[0][1].w_in.n, dtype=bf, device=dev)
    q, attn = torch.randn(t, m.heads, m.dim, dtype=bf, device=dev), torch.randn(t, m.heads, m.vdim, dtype=bf, device=dev)
    cos = torch.ones(t, m.dim // 2, device=dev)
    qkv = raw[:, :nq + 2 * nkv].contiguous()
    tab.add(ph, "window: q|k|v|gate projection", [lambda w=w: N.linear(h, w.w_in.w, raw) for _, w, _ in win],
            gemm(nq + 2 * nkv, d), "qkv projection", [lambda w=w: gemm_bf16(h, w.w_in.w[:nq + 2 * nkv], out=qkv) for _, w, _ in win])
    tab.add(ph, "window: head norms + append", [lambda i=i, w=w: N.head_norm_append(
        raw, w.q_norm, w.k_norm, 1e-6, q, cache.k[i], cache.v[i], c.block_table, c.positions, c.token_seq, m.heads, m.dim,
        m.vdim) for i, w, _ in win], (t * (nq + 2 * nkv) * 4, 0), "rope + append",
        [lambda i=i: D.rope_kv_write(qkv, q, cache.k[i], cache.v[i], c.block_table, c.positions, cos, cos, m.heads, m.kv_heads,
                                     token_seq=c.token_seq) for i, _, _ in win])
    seen = sum(min(p + 1, WINDOW) for p in range(t))
    cost = (t * (2 * nq + 2 * nkv) * 2, 4.0 * m.heads * m.dim * seen)
    gate = raw[:, win[0][1].gate_at:win[0][1].gate_at + m.heads]
    tab.add(ph, "window: attention + gate", [lambda i=i, w=w: P.flash_prefill_scored(
        q, cache.k[i], cache.v[i], c.block_table, batch.tiles, w.mods, attn, window=m.window, lanes=batch.lanes, gate=gate)
        for i, w, _ in win], cost, "attention, same window",
        [lambda i=i: flash_prefill_paged(q, cache.k[i], cache.v[i], row, 0, m.scale, window=WINDOW) for i, _, _ in win])
    # output projection, norm
    a2 = attn.view(t, -1)
    tab.add(ph, "output projection", [lambda w=w: P.logits_f32(a2, w.w_o.w, y) for _, w, _ in win], gemm(d, nq, 4),
            "o projection + residual", [lambda w=w: gemm_bf16(a2, w.w_o.w, residual=res, out=h) for _, w, _ in win],
            gemm(d, nq, 4))
    tab.add(ph, "output norm + residual", [lambda l=l: N.post_norm_add(y, l.norm1, 1e-6, d, x, h) for l in model.w.layers],
            (t * d * 14, 0), "norm", [lambda l=l: D.rms_norm(h, res[0], 1e-6) for l in model.w.layers], (t * d * 4, 0))
    # dense feed-forward
    f = dense[0][1]
    ff = f.w_down.k
    act = torch.randn(t, ff, dtype=bf, device=dev)
    tab.add(ph, "dense: gate/up + activation", [lambda w=w: N.gated_linear(h, w.w_gu, 7.0, act, None) for _, w, _ in dense],
            (2 * ff * d * 2 + t * (d + ff) * 2, 4.0 * t * d * ff), "gate/up + SwiGLU",
            [lambda w=w: xgemm(h, w.w_gu, out=act, swiglu=True) for _, w, _ in dense])
    tab.add(ph, "dense: down", [lambda w=w: P.logits_f32(act, w.w_down.w, y) for _, w, _ in dense], gemm(d, ff, 4),
            "down + residual", [lambda w=w: gemm_bf16(act, w.w_down.w, residual=res, out=h) for _, w, _ in dense], gemm(d, ff, 4))
    del act
    # routed
    f = moe[0][1]
    ex, pairs, outs = f.w_down.k, t * TOP, EXPERTS + IDENTITY
    z, z_out = torch.randn(t, outs, device=dev), torch.empty(t, outs, device=dev)
    r = model.routing(f, c)
    R.route_corrected(z, f.correction, EXPERTS, r)
    xs = torch.randn(pairs, d, dtype=bf, device=dev)
    R.route_scatter(h, r, xs)
    used = int(r.offsets[-1])
    offs = r.offsets.clone()
    act, ye = torch.randn(pairs, ex, dtype=bf, device=dev), torch.randn(pairs, d, dtype=bf, device=dev)
    idx = torch.randint(0, EXPERTS, (t, TOP), dtype=torch.int32, device=dev)
    z32 = torch.randn(t, EXPERTS, device=dev)
    counts, offs2 = torch.zeros(EXPERTS, dtype=torch.int32, device=dev), torch.zeros(EXPERTS + 1, dtype=torch.int32, device=dev)
    wts = torch.rand(t, TOP, device=dev)
    from rmlx_b200 import _lib
    lib = _lib.cuda()
    tab.add(ph, "routed: router logits", [lambda w=w: P.logits_f32(h, w.router, z_out) for _, w, _ in moe], gemm(outs, d, 4))

    def route_like():
        lib.rmlx_topk_route(z32.data_ptr(), None, idx.data_ptr(), wts.data_ptr(), counts.data_ptr(), offs2.data_ptr(), t, EXPERTS,
                            TOP, _lib.stream_ptr())
    tab.add(ph, "routed: choice + offsets", [lambda: R.route_corrected(z, f.correction, EXPERTS, r) for _ in moe],
            (t * (outs * 4 + TOP * 8 + 4), 0), "top-k route + offsets", [route_like for _ in moe], (t * (EXPERTS * 4 + TOP * 8), 0))
    cursors, rows2 = torch.zeros(EXPERTS, dtype=torch.int32, device=dev), torch.zeros(t, TOP, dtype=torch.int32, device=dev)

    def scatter():                         # the same choice as above: ``offs`` are its row ranges
        r.counts.copy_(offs[:-1])
        R.route_scatter(h, r, xs)

    def scatter_like():
        lib.rmlx_moe_scatter_rows(h.data_ptr(), d, idx.data_ptr(), offs2.data_ptr(), cursors.data_ptr(), xs.data_ptr(),
                                  rows2.data_ptr(), t, TOP, d, EXPERTS, _lib.stream_ptr())
    route_like()
    scatter_like()
    tab.add(ph, "routed: scatter", [scatter for _ in moe], ((t + used) * d * 2, 0), "scatter", [scatter_like for _ in moe],
            ((t + pairs) * d * 2, 0))
    tab.add(ph, "routed: experts' gate/up", [lambda w=w: xgemm(xs, w.w_gu, offsets=offs, out=act, swiglu=True, gate_limit=7.0)
                                             for _, w, _ in moe],
            (EXPERTS * 2 * ex * d * 2 + used * (d + ex) * 2, 4.0 * used * d * ex), "experts' gate/up + SwiGLU",
            [lambda w=w: xgemm(xs, w.w_gu, offsets=offs2, out=act, swiglu=True) for _, w, _ in moe],
            (EXPERTS * 2 * ex * d * 2 + pairs * (d + ex) * 2, 4.0 * pairs * d * ex))
    tab.add(ph, "routed: experts' down", [lambda w=w: xgemm(act, w.w_down, offsets=offs, out=ye) for _, w, _ in moe],
            (EXPERTS * ex * d * 2 + used * (d + ex) * 2, 2.0 * used * d * ex), "experts' down",
            [lambda w=w: xgemm(act, w.w_down, offsets=offs2, out=ye) for _, w, _ in moe],
            (EXPERTS * ex * d * 2 + pairs * (d + ex) * 2, 2.0 * pairs * d * ex))

    def combine_like():
        lib.rmlx_moe_combine(ye.data_ptr(), rows2.data_ptr(), wts.data_ptr(), res.data_ptr(), d, h.data_ptr(), d, t, TOP, d,
                             _lib.stream_ptr())
    tab.add(ph, "routed: combine + norm + residual", [lambda l=l: R.combine_post_norm(ye, r, l.norm2, 1e-6, d, x, h)
                                                      for _, _, l in moe], (used * d * 2 + t * d * 10, 0), "combine + residual",
            [combine_like for _ in moe], (pairs * d * 2 + t * d * 4, 0))
    del xs, act, ye
    # latent attention
    m = lat[0][1].spec
    w0 = lat[0][1]
    raw = torch.randn(t, w0.w_in.n, dtype=bf, device=dev)
    q = torch.randn(t, m.heads, w0.dim_p + w0.rot_p, dtype=bf, device=dev)
    attn = torch.randn(t, m.heads, w0.vdim_p, dtype=bf, device=dev)
    q_like = torch.empty(t, m.heads, 128, dtype=bf, device=dev)
    ctx, kv = torch.randn(t, w0.lat_p, dtype=bf, device=dev), torch.randn(t, m.heads, w0.dim_p + w0.vdim_p, dtype=bf, device=dev)
    n_in, n_kv = w0.w_in.n, kv.shape[1] * kv.shape[2]
    tab.add(ph, "latent: q|latent projection", [lambda w=w: N.linear(h, w.w_in.w, raw) for _, w, _ in lat], gemm(n_in, d),
            "the same GEMM", [lambda w=w: gemm_bf16(h, w.w_in.w, out=raw) for _, w, _ in lat])
    tab.add(ph, "latent: norm + rotation + append", [lambda i=i, w=w: N.latent_append(
        raw, raw[:, w.down_at:], w.c_norm, 1e-6, w.inv_freq, q, None, cache.k[i], c.block_table, c.positions, c.token_seq, m.heads, m.dim, m.rot_dim,
        m.kv_rank, w.dim_p, w.rot_p, w.lat_p) for i, w, _ in lat], (t * n_in * 4, 0), "rope + append",
        [lambda: D.rope_kv_write(qkv, q_like, cache.k[win[0][0]], cache.v[win[0][0]], c.block_table, c.positions, cos, cos,
                                 m.heads, win[0][1].spec.kv_heads, token_seq=c.token_seq) for _ in lat],
        (t * qkv.shape[1] * 4, 0))
    tab.add(ph, "latent: gather", [lambda i=i: L.latent_gather(cache.k[i], c.block_table, batch.ctx_pages, ctx) for i, _, _ in lat],
            (t * w0.lat_p * 4, 0))
    tab.add(ph, "latent: expand keys and values", [lambda w=w: N.linear(ctx, w.w_ukv.w, kv.view(t, -1)) for _, w, _ in lat],
            gemm(n_kv, w0.lat_p))
    cost = (t * m.heads * (192 + 128 + 256) * 2, 2.0 * m.heads * (m.dim + m.rot_dim + m.vdim) * t * (t + 1) / 2)
    q128 = torch.randn(t, m.heads, 128, dtype=bf, device=dev)
    kc = torch.randn(t // 16 + 2, m.heads, 16, 128, dtype=bf, device=dev)
    vc = torch.randn_like(kc)
    tab.add(ph, "latent: attention", [lambda i=i: L.flash_prefill_latent(
        q, kv, cache.k[i], w0.lat_p, c.block_table, batch.latent_tiles, batch.tile_ctx, m.scale, attn, w0.dim_p,
        lanes=batch.latent_lanes) for i, _, _ in lat], cost, "attention, as many heads",
        [lambda: flash_prefill_paged(q128, kc, vc, row, 0, m.scale) for _ in lat],
        (t * m.heads * 512 * 2, 4.0 * m.heads * 128 * t * (t + 1) / 2))
    del raw, q, attn, ctx, kv, q128, kc, vc
    # WKV
    m = wkv[0][1].spec
    w0 = wkv[0][1]
    inner = w0.inner_p
    mix = torch.randn(5, t, d, dtype=bf, device=dev)
    rkvg = torch.randn(4, t, inner, dtype=bf, device=dev)
    decay, o = torch.randn(t, inner, device=dev), torch.randn(t, inner, device=dev)
    a = torch.randn(t, inner, dtype=bf, device=dev)
    st = lambda i: (cache.layer_state(i, "wkv"), cache.layer_state(i, "prev"))               # noqa: E731
    tab.add(ph, "wkv: token shift", [lambda i=i, w=w: W.token_shift(x, w.mu, st(i)[1], c.slots, False, mix) for i, w, _ in wkv],
            (t * d * (4 + 10), 0))
    tab.add(ph, "wkv: one of r, k, v, g", [lambda w=w: N.linear(mix[0], w.part(0), rkvg[0]) for _, w, _ in wkv], gemm(inner, d),
            "the same GEMM", [lambda w=w: gemm_bf16(mix[0], w.part(0), out=rkvg[0]) for _, w, _ in wkv])
    low, low_t = torch.randn(t, w0.rank_p, device=dev), torch.randn(t, w0.rank_p, dtype=bf, device=dev)
    tab.add(ph, "wkv: decay, first factor", [lambda w=w: P.logits_f32(mix[4], w.part(4), low) for _, w, _ in wkv], gemm(w0.rank_p, d, 4))
    tab.add(ph, "wkv: decay, second factor", [lambda w=w: P.logits_f32(low_t, w.w2, decay) for _, w, _ in wkv],
            gemm(inner, w0.rank_p, 4))
    rec = torch.empty(t * m.heads * W.record(m.dim), device=dev)
    tab.add(ph, "wkv: recurrence", [lambda i=i, w=w: W.wkv_scan(rkvg[0], rkvg[1], rkvg[2], decay, w.w0, w.u, *st(i), x, o, rec,
                                                                runs=batch.runs) for i, w, _ in wkv],
            (t * inner * (6 + 4 + 4), 0, 3.0 * t * inner * m.dim))
    tab.add(ph, "wkv: head norm + gate", [lambda w=w: W.wkv_finish(o, rkvg[3], w.norm, 1e-6, m.heads, m.dim, a) for _, w, _ in wkv],
            (t * inner * 8, 0))


def decode_kernels(tab: Table, model: RodapelModel, b: int, ctx: int):
    cfg, d, dev, bf = model.cfg, model.cfg.width, model.device, torch.bfloat16
    win, lat, wkv, dense, moe = kinds(model)
    cache = filled_cache(model, b, ctx, 32)
    eng = model.make_decode_engine(cache, b)
    eng.bind(list(range(b)), [1] * b)
    eng.reserve(4)
    if not (eng.fused and b <= eng.matvec_rows):
        return
    c = eng._context(b)
    ph = f"decode b{b} ctx {ctx}"
    x, x2, y = (torch.randn(b, d, device=dev) for _ in range(3))
    h, res = torch.randn(b, d, dtype=bf, device=dev), torch.randn(b, d, dtype=bf, device=dev)
    nw = torch.ones(d, dtype=bf, device=dev)
    pend = lambda l: N.Pending(y, l.norm1)                                                   # noqa: E731
    m = win[0][1].spec
    nq, nkv = m.heads * m.dim, m.kv_heads * m.dim
    w0 = win[0][1]
    raw = torch.randn(b, w0.w_in.n, device=dev)
    out16 = torch.empty(b, w0.w_in.n, dtype=bf, device=dev)
    tab.add(ph, "window: output norm + q|k|v|gate", [lambda w=w, l=l: N.postnorm_in(x, pend(l), 1e-6, d, x2, w.w_in.w, raw, pdl=True)
                                                     for _, w, l in win], (w0.w_in.n * d * 2, 0), "norm + projection",
            [lambda w=w: D.rms_gemv(h, w.w_in, nw, 1e-6, out=out16, pdl=True) for _, w, _ in win])
    attn = torch.randn(b, m.heads, m.vdim, dtype=bf, device=dev)
    q16 = torch.randn(b, m.heads, m.dim, dtype=bf, device=dev)
    scr = model.scratch(m.heads, m.kv_heads, m.vdim, b, model.attention_splits(m, b, c.max_len, m.window))
    from rmlx_b200 import _lib
    gt = _lib.cuda().rmlx_flash_decode_gtiles(m.heads, m.kv_heads)
    sp = D.default_splits(b, m.kv_heads, gt, WINDOW)
    fd = D.FlashDecodeScratch(b, m.heads, m.kv_heads, m.dim, sp, dev, max_len=c.max_len)
    kv = b * min(ctx, WINDOW) * 2 * nkv * 2
    tab.add(ph, "window: head norms + append + attention + gate", [lambda i=i, w=w: P.flash_decode_scored(
        cache.k[i], cache.v[i], c.block_table, c.positions, w.mods, attn, scr, m.heads, m.dim, m.vdim, raw=raw, q_w=w.q_norm,
        k_w=w.k_norm, eps=1e-6, n_rows=b, window=m.window, head_norm=True, gate_col=w.gate_at, pdl=True) for i, w, _ in win],
        (kv, 0), "attention, same window", [lambda i=i: D.flash_decode_paged(
            q16, cache.k[i], cache.v[i], c.block_table, eng.seq_lens, m.scale, sp, fd, WINDOW, out=attn, pdl=True)
            for i, _, _ in win])
    a2 = attn.view(b, -1)
    tab.add(ph, "output projection", [lambda w=w: N.matvec_out(a2, w.w_o.w, y, pdl=True) for _, w, _ in win], (nq * d * 2, 0),
            "o projection + residual", [lambda w=w: D.rms_gemv(a2, w.w_o, None, 1e-6, residual=res, out=h, pdl=True)
                                        for _, w, _ in win])
    f = dense[0][1]
    ff = f.w_down.k
    act = torch.randn(b, ff, dtype=bf, device=dev)
    tab.add(ph, "dense: output norm + gate/up + activation", [lambda w=w, l=l: N.postnorm_gated(
        x, pend(l), 1e-6, d, x2, w.w_gu.w, 7.0, act, pdl=True) for _, w, l in dense], (2 * ff * d * 2, 0),
        "norm + gate/up + SwiGLU", [lambda w=w: D.rms_gate_up_swiglu(h, w.w_gu, nw, 1e-6, out=act, pdl=True) for _, w, _ in dense])
    tab.add(ph, "dense: down", [lambda w=w: N.matvec_out(act, w.w_down.w, y, pdl=True) for _, w, _ in dense], (ff * d * 2, 0),
            "down + residual", [lambda w=w: D.rms_gemv(act, w.w_down, None, 1e-6, residual=res, out=h, pdl=True)
                                for _, w, _ in dense])
    f = moe[0][1]
    ex, outs = f.w_down.k, EXPERTS + IDENTITY
    r = model.routing(f, c)
    z = torch.randn(b, outs, device=dev)
    rs = D.RouterScratch(b, EXPERTS, dev)
    idx, wts = torch.zeros(b, TOP, dtype=torch.int32, device=dev), torch.rand(b, TOP, device=dev)
    tab.add(ph, "routed: output norm + router + choice", [lambda w=w, l=l: R.postnorm_router(
        x, pend(l), 1e-6, d, x2, w.router, w.correction, EXPERTS, z, eng.ticket, r, pdl=True) for _, w, l in moe],
        (outs * d * 2, 0), "norm + router + top-k", [lambda w=w: D.moe_router(h, w.router[:EXPERTS], nw, 1e-6, TOP, None, rs, idx,
                                                                             wts, pdl=True) for _, w, _ in moe],
        (EXPERTS * d * 2, 0))
    for i in range(b):                     # fixed, distinct experts: every slot has work
        r.idx[i] = torch.arange(i * TOP, (i + 1) * TOP, dtype=torch.int32) % EXPERTS
    r.weights.fill_(0.25)
    r.identity.zero_()
    idx.copy_(r.idx)
    acte = torch.randn(b * TOP, ex, dtype=bf, device=dev)
    tab.add(ph, "routed: experts' gate/up", [lambda w=w: R.postnorm_expert(x, w.w_gu.w, 7.0, r, acte, pdl=True) for _, w, _ in moe],
            (b * TOP * 2 * ex * d * 2, 0), "norm + experts' gate/up + SwiGLU",
            [lambda w=w: D.moe_gate_up(h, w.w_gu, nw, 1e-6, idx, out=acte, pdl=True) for _, w, _ in moe])
    tab.add(ph, "routed: experts' down + identity", [lambda w=w: R.expert_out(acte, w.w_down.w, r, x, y, pdl=True) for _, w, _ in moe],
            (b * TOP * ex * d * 2, 0), "experts' down + residual",
            [lambda w=w: D.moe_down(acte, w.w_down, idx, wts, residual=res, out=h, pdl=True) for _, w, _ in moe])
    m, w0 = lat[0][1].spec, lat[0][1]
    raw = torch.randn(b, w0.w_in.n, device=dev)
    out16 = torch.empty(b, w0.w_in.n, dtype=bf, device=dev)
    tab.add(ph, "latent: output norm + q|latent", [lambda w=w, l=l: N.postnorm_in(x, pend(l), 1e-6, d, x2, w.w_in.w, raw, pdl=True)
                                                   for _, w, l in lat], (w0.w_in.n * d * 2, 0), "norm + projection",
            [lambda w=w: D.rms_gemv(h, w.w_in, nw, 1e-6, out=out16, pdl=True) for _, w, _ in lat])
    q = torch.randn(b, m.heads, w0.dim_p + w0.rot_p, dtype=bf, device=dev)
    q_abs = torch.randn(b, m.heads, w0.lat_p + w0.rot_p, dtype=bf, device=dev)
    o_lat, attn = torch.randn(b, m.heads, w0.lat_p, dtype=bf, device=dev), torch.randn(b, m.heads, w0.vdim_p, dtype=bf, device=dev)
    tab.add(ph, "latent: norm + rotation + append", [lambda i=i, w=w: N.latent_append(
        raw, raw[:, w.down_at:], w.c_norm, 1e-6, w.inv_freq, q, q_abs, cache.k[i], c.block_table, c.positions, None, m.heads, m.dim, m.rot_dim,
        m.kv_rank, w.dim_p, w.rot_p, w.lat_p, pdl=True) for i, w, _ in lat], (b * w0.w_in.n * 6, 0))
    tab.add(ph, "latent: queries into the latent space", [lambda w=w: N.head_gemv(w.w_uk, q, q_abs, pdl=True) for _, w, _ in lat],
            (w0.w_uk.numel() * 2, 0), "einsum (as the latent-attention model)",
            [lambda w=w: torch.einsum("bhd,hld->bhl", q[..., :w0.dim_p], w.w_uk) for _, w, _ in lat])
    scr = L.LatentDecodeScratch(b, m.heads, L.decode_splits(b, m.heads, c.max_len), w0.lat_p, dev)
    tab.add(ph, "latent: attention (the framework's kernel)", [lambda i=i: L.latent_decode(
        q_abs, cache.k[i], c.block_table, c.positions, m.scale, o_lat, scr, pdl=True) for i, _, _ in lat],
        (b * ctx * (w0.lat_p + w0.rot_p + 8) * 2, 0))
    tab.add(ph, "latent: values", [lambda w=w: N.head_gemv(w.w_uv, o_lat, attn, pdl=True) for _, w, _ in lat],
            (w0.w_uv.numel() * 2, 0), "einsum (as the latent-attention model)",
            [lambda w=w: torch.einsum("bhl,hvl->bhv", o_lat, w.w_uv) for _, w, _ in lat])
    m, w0 = wkv[0][1].spec, wkv[0][1]
    raw = torch.randn(b, w0.w_in.n, device=dev)
    out16 = torch.empty(b, w0.w_in.n, dtype=bf, device=dev)
    st = lambda i: (cache.layer_state(i, "wkv"), cache.layer_state(i, "prev"))               # noqa: E731
    tab.add(ph, "wkv: output norm + shift + projections", [lambda i=i, w=w, l=l: N.postnorm_in(
        x, pend(l), 1e-6, d, x2, w.w_in.w, raw, shift=(w.mu, st(i)[1], c.slots, w.inner_p), pdl=True) for i, w, l in wkv],
        (w0.w_in.n * d * 2, 0), "norm + projection", [lambda w=w: D.rms_gemv(h, w.w_in, nw, 1e-6, out=out16, pdl=True)
                                                      for _, w, _ in wkv])
    a = torch.randn(b, w0.inner_p, dtype=bf, device=dev)
    tab.add(ph, "wkv: decay + recurrence + head norm + gate", [lambda i=i, w=w: W.wkv_decode(
        raw, w.inner_p, w.w2, w.w0, w.u, w.norm, 1e-6, c.slots, *st(i), x, a, pdl=True) for i, w, _ in wkv],
        (w0.w2.numel() * 2 + b * m.heads * m.dim * m.dim * 8, 0))


def main(argv=None) -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--sizes", default="2048,4096")
    ap.add_argument("--layers", type=int, default=8)
    ap.add_argument("--tokens", default="2048,8192")
    ap.add_argument("--batches", default="1,8,64")
    ap.add_argument("--ctx", type=int, default=4096)
    ap.add_argument("--kernels", action="store_true", help="also every kernel against its roofline")
    a = ap.parse_args(argv)
    tokens, batches = [int(x) for x in a.tokens.split(",")], [int(x) for x in a.batches.split(",")]
    dev = torch.device("cuda:0")
    for width in (int(x) for x in a.sizes.split(",")):
        cfg = rodapel_cfg(width, a.layers)
        model = RodapelModel(build_weights(cfg, random_tensors(cfg, 0, dev), dev))
        ours = run_models(model, tokens, batches, a.ctx)
        if a.kernels:
            with torch.no_grad():
                for t in tokens:
                    prefill_kernels(Table(width), model, t)
                    torch.cuda.empty_cache()
                for b in batches:
                    decode_kernels(Table(width), model, b, a.ctx)
                    torch.cuda.empty_cache()
            GemmStatus.check(dev)
        nbytes = model.w.nbytes()
        del model
        torch.cuda.empty_cache()
        max_len = max(max(tokens), a.ctx + 128)
        model = TransformerModel(random_on_device(moe_cfg(width, a.layers, max_len), dev, None))
        moe = run_models(model, tokens, batches, a.ctx)
        print(json.dumps({"width": width, "layers": a.layers, "ctx": a.ctx, "unit": "tokens/s", "rodapel": ours,
                          "moe_transformer": moe, "weight_bytes": [nbytes, model.w.nbytes()],
                          "ratio": {k: round(ours[k] / moe[k], 3) for k in ours if ours[k] and moe[k]}}), flush=True)
        del model
        torch.cuda.empty_cache()
    return 0


if __name__ == "__main__":
    sys.exit(main())
