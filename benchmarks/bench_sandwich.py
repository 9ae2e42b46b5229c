#!/usr/bin/env python
"""Prefill and decode throughput of the sandwich-norm decoder (Nizorax) beside the framework's closest model, the post-norm
decoder (Rodapel), at equal size, and its new kernels beside the like kernels of the framework's other models, each against
its roofline. Random weights, one GPU, bf16.

    python benchmarks/bench_sandwich.py [--sizes 2048,4096] [--layers 8] [--kernels]
    python bench.py --suite sandwich ...       # the same

Layers come in fours: windowed differential attention + dense, lightning attention + routed (twice), windowed differential
attention + routed. Equal size: the post-norm decoder has windowed attention and WKV in their places, the same width, heads
(128 query values and 128 value channels each), window, expert count and width, as many experts per token (its fifth one is
routed, here it is the shared one) and as many dense weights. Prefill: one prompt of ``--tokens``; decode: B sequences of
``--ctx`` cached tokens, one captured step per token. Timing: CUDA events after warm-up; the layers' weights together exceed
L2. Kernel times: graph-captured loops over all layers of a kind (each with its own weights and pages). "roofline" is the
largest of bytes / copy bandwidth, tensor FLOPs / burst GEMM rate (MEASURED_PEAKS.json) and, for the recurrences, fp32
operations / (SMs x 128 a clock at the top clock)."""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
from bench_parallel_block import VOCAB  # noqa: E402
from bench_post_norm import EXPERTS, HD, SIZES, TOP, WINDOW, Table, filled_cache, run_models  # noqa: E402
from bench_twin_norm import WkvLike  # noqa: E402

from rmlx_b200.config import (ClampedFfSpec, DifferentialAttentionSpec, GroupedFfSpec, LightningSpec, NizoraxConfig,  # noqa: E402
                              PolyNormFfSpec, PostNormLayerSpec, RodapelConfig, RotarySpec, RoutedFfSpec, SandwichLayerSpec,
                              WindowAttentionSpec, WkvSpec)
from rmlx_b200.models import rodapel  # noqa: E402
from rmlx_b200.models.nizorax import (DiffAttentionWeights, LightningWeights, NizoraxModel, PolyFfWeights,  # noqa: E402
                                      build_weights, random_tensors)
from rmlx_b200.models.ragged import Entry, RaggedBatch  # noqa: E402
from rmlx_b200.models.ragged_model import Buffers, DenseFfWeights, RoutedFfWeights, StepContext  # noqa: E402
from rmlx_b200.ops import parallel_block as P  # noqa: E402
from rmlx_b200.ops import post_norm as N  # noqa: E402
from rmlx_b200.ops import routed as R  # noqa: E402
from rmlx_b200.ops import sandwich as W  # noqa: E402
from rmlx_b200.ops import scan as S  # noqa: E402
from rmlx_b200.ops import twin_norm as TN  # noqa: E402
from rmlx_b200.ops import wkv  # noqa: E402
from rmlx_b200.ops.gemm import GemmStatus  # noqa: E402

BF, F32 = torch.bfloat16, torch.float32
GROUPS, KEEP, TAPS = 8, 4, 4


def nizorax_cfg(width: int, layers: int) -> NizoraxConfig:
    hq, hkv, inner, ex = SIZES[width]
    rot = RotarySpec(500000.0, 64, {"factor": 8.0, "original": 8192.0, "high": 4.0, "low": 1.0})
    attn = DifferentialAttentionSpec(hq, hkv, HD // 2, HD, (HD // 2) ** -0.5, rot, 0.4, WINDOW)
    heads = width // 128
    light = LightningSpec(heads, 128, 128, [1.0 - 2.0 ** (-1 - 8 * i / heads) for i in range(heads)])
    moe = GroupedFfSpec(EXPERTS, TOP, ex, GROUPS, KEEP, 1.0, ex)
    four = [SandwichLayerSpec(attn, PolyNormFfSpec(inner * 3 // 2)), SandwichLayerSpec(light, moe), SandwichLayerSpec(light, moe),
            SandwichLayerSpec(attn, moe)]
    return NizoraxConfig(VOCAB, width, four * (layers // 4), 1e-6, taps=TAPS).validate()


def like_cfg(width: int, layers: int) -> RodapelConfig:
    hq, hkv, inner, ex = SIZES[width]
    win = WindowAttentionSpec(hq, hkv, HD, HD, HD ** -0.5, WINDOW)
    moe, rec = RoutedFfSpec(EXPERTS, 0, TOP + 1, ex, 7.0), WkvSpec(width // 64, 64, 64)
    four = [PostNormLayerSpec(win, ClampedFfSpec(inner, 7.0)), PostNormLayerSpec(rec, moe), PostNormLayerSpec(rec, moe),
            PostNormLayerSpec(win, moe)]
    return RodapelConfig(VOCAB, width, four * (layers // 4), 1e-6).validate()


def kinds(model):
    ls = list(enumerate(model.w.layers))
    pick = lambda cls, part: [(i, getattr(l, part), l) for i, l in ls if isinstance(getattr(l, part), cls)]   # noqa: E731
    return (pick(DiffAttentionWeights, "mix"), pick(LightningWeights, "mix"), pick(PolyFfWeights, "mlp"), pick(RoutedFfWeights, "mlp"))


def prefill_kernels(tab: Table, model: NizoraxModel, like, t: int):
    cfg, d, dev = model.cfg, model.cfg.width, model.device
    attn_ls, light, dense, moe = kinds(model)
    like_moe = [l.mlp for l in like.w.layers if isinstance(l.mlp, RoutedFfWeights)]
    cache = model.new_cache(t // 16 + 2, max_seqs=1, max_blocks_per_seq=t // 16 + 1)
    cache.add_sequence(0)
    batch = RaggedBatch.plan([Entry(0, [1] * t)], cache, 0)
    cache.reserve(0, t)
    batch.upload(dev)
    c = StepContext(t, Buffers(t, dev), cache, cache.block_table, batch.positions, batch.token_seq, batch.token_seq, batch.runs, batch)
    for pool in {id(p): p for p in cache.k + cache.v if p is not None}.values():
        pool.normal_()
    rnd = lambda *s, dtype=BF: torch.randn(*s, device=dev, dtype=dtype)                      # noqa: E731
    x, h, y, y32, hc = rnd(t, d, dtype=F32), rnd(t, d), rnd(t, d), rnd(t, d, dtype=F32), rnd(t, d)
    ph, each, one = f"prefill {t}", list(enumerate(model.w.layers)), torch.ones(d, device=dev)
    gemm = lambda n, k, out=2: (n * k * 2 + t * (k * 2 + n * out), 2.0 * t * n * k)          # noqa: E731
    norm_like = [lambda: N.post_norm_add(y32, one, 1e-6, d, x, h) for _ in each]
    tab.add(ph, "output norm + residual + norm", [lambda l=l: W.sandwich_norm(x, y, l.post1, l.norm2, h, 1e-6, d) for _, l in each],
            (t * d * 12, 0), "output norm + residual", norm_like, (t * d * 14, 0))
    mu, prev, mix = torch.rand(5, d, device=dev), torch.zeros(2, d, device=dev), torch.empty(5, t, d, dtype=BF, device=dev)
    tab.add(ph, "short convolution", [lambda i=i, l=l: W.short_conv(h, l.conv1, cache.layer_state(i, "conv1"), hc, c.slots, runs=c.runs)
                                      for i, l in each], (t * d * 4, 0), "token shift", [lambda: wkv.token_shift(
                                          x, mu, prev, c.slots, False, mix) for _ in each], (t * d * 14, 0))
    del mix
    # attention
    w0 = attn_ls[0][1]
    m = w0.spec
    raw = rnd(t, w0.w_in.n)
    q, out = rnd(t, m.heads, 2, m.dim), rnd(t, m.heads, m.vdim)
    rows = (m.heads + m.kv_heads) * 2 * m.dim + m.kv_heads * m.vdim
    table = (c.block_table, c.positions, c.token_seq)
    q1, ones = q.view(t, m.heads, HD), torch.ones(HD, device=dev)
    tab.add(ph, "attention: rotation + append", [lambda i=i, w=w: TN.rotary_norm_append(
        raw, None, w.inv_freq, 1.0, 0.0, q, cache.k[i], cache.v[i], *table, m.heads, m.dim, m.vdim, neighbours=True, norm=False,
        maps=2) for i, w, _ in attn_ls], (t * rows * 4, 0), "head norms + append", [lambda i=i: N.head_norm_append(
            raw, ones, ones, 1e-6, q1, cache.k[i], cache.v[i], *table, m.heads, HD, HD) for i, _, _ in attn_ls])
    seen = sum(min(p + 1, WINDOW) for p in range(t))
    nq = m.heads * HD
    batch2 = RaggedBatch.plan([Entry(0, [1] * t)], cache, m.heads).upload(dev)
    tab.add(ph, "attention: two maps, difference, norm", [lambda i=i, w=w: P.flash_prefill_diff(
        q, cache.k[i], cache.v[i], c.block_table, batch.tiles, w.mods.scale, w.diff, m.vdim, out, window=WINDOW)
        for i, w, _ in attn_ls], (t * (2 * nq + 2 * m.kv_heads * HD) * 2, 2.0 * m.heads * (2 * m.dim + 2 * m.vdim) * seen),
        "attention, same window", [lambda i=i, w=w: P.flash_prefill_scored(
            q1, cache.k[i], cache.v[i], c.block_table, batch2.tiles, w.mods, out, window=WINDOW, lanes=batch2.lanes)
            for i, w, _ in attn_ls], (t * (2 * nq + 2 * m.kv_heads * HD) * 2, 4.0 * m.heads * HD * seen))
    del raw, q, q1, out
    # lightning
    g0 = light[0][1]
    m = g0.spec
    raw = rnd(t, g0.w_in.n)
    o, a = torch.empty(t, g0.w_o.k, device=dev), torch.empty(t, g0.w_o.k, dtype=BF, device=dev)
    rec = torch.empty(t * m.heads * S.record(m.dim, m.vdim, True), device=dev)
    q, k, v, g = (raw[:, at:] for at in g0.at)
    like_rec = WkvLike(d, t, dev)
    tab.add(ph, "lightning: recurrence", [lambda i=i, w=w: S.lightning_scan(
        q, k, v, w.decay, cache.layer_state(i, "state"), o, rec, runs=batch.runs) for i, w, _ in light],
        (t * m.heads * (2 * m.dim + 3 * m.vdim) * 2, 0, 3.0 * t * m.heads * m.dim * m.vdim), "WKV recurrence",
        [lambda: like_rec.scan(batch.runs) for _ in light], (t * d * 14, 0, 3.0 * t * d * 64))
    tab.add(ph, "lightning: norm + gate", [lambda w=w: S.gated_norm(o, g, w.norm, 1e-6, 1, a, False, sigmoid=True) for _, w, _ in light],
            (t * g0.w_o.k * 8, 0), "head norm + gate", [lambda: wkv.wkv_finish(
                like_rec.o, like_rec.r, like_rec.w0, 1e-6, like_rec.h, 64, a[:, :d]) for _ in light], (t * d * 8, 0))
    del raw, rec, o, a, like_rec
    # dense feed-forward
    f = dense[0][1]
    ff = f.w_up.n
    z = rnd(t, ff)
    tab.add(ph, "dense: up projection", [lambda w=w: N.linear(hc, w.w_up.w, z) for _, w, _ in dense], gemm(ff, d))
    half = torch.empty(t, ff // 2, dtype=BF, device=dev)
    tab.add(ph, "dense: polynomial of normed powers", [lambda w=w: W.poly_norm(z, w.act, 1e-6, f.spec.ff, z) for _, w, _ in dense],
            (t * ff * 4, 0), "gated activation", [lambda: N.gated_act(z, half, 7.0) for _ in dense], (t * ff * 3, 0))
    tab.add(ph, "dense: down projection", [lambda w=w: N.linear(z, w.w_down.w, y) for _, w, _ in dense], gemm(d, ff))
    del z, half
    # routed
    f = moe[0][1]
    slots, ex = TOP + f.always, f.w_down.k
    zr = rnd(t, EXPERTS, dtype=F32)
    r, lr = model.routing(f, c), like.routing(like_moe[0], StepContext(t, Buffers(t, dev), cache, None, None, None, None, None))
    tab.add(ph, "routed: choice + offsets", [lambda: R.route_grouped(zr, model.groups(f), r) for _ in moe],
            (t * (EXPERTS * 4 + slots * 8), 0), "corrected choice + offsets",
            [lambda: R.route_corrected(zr, like_moe[0].correction, EXPERTS, lr) for _ in moe])
    xs, xs2 = torch.empty(t * slots, d, dtype=BF, device=dev), torch.empty(t * slots, d, dtype=BF, device=dev)

    def scatter(routing, to, always, choose):             # the cursors are used up: the choice belongs to it
        choose()
        R.route_scatter(h, routing, to, always)

    tab.add(ph, "routed: choice + scatter", [lambda: scatter(r, xs, f.always, lambda: R.route_grouped(zr, model.groups(f), r))
                                             for _ in moe], (t * d * 2 * (slots + 1), 0), "corrected choice + scatter",
            [lambda: scatter(lr, xs2, 0, lambda: R.route_corrected(zr, like_moe[0].correction, EXPERTS, lr)) for _ in moe])
    del xs2
    act, ye = rnd(t * slots, ex), rnd(t * slots, d)
    cost = ((EXPERTS + f.always) * 3 * ex * d * 2 + t * slots * (2 * d + 2 * ex) * 2, 6.0 * t * slots * ex * d)
    R.route_grouped(zr, model.groups(f), r)
    offs = r.offsets.clone()
    R.route_corrected(zr, like_moe[0].correction, EXPERTS, lr)
    loffs = lr.offsets.clone()
    tab.add(ph, "routed: experts and shared expert", [lambda w=w: R.grouped_gated_ffn(xs, offs, w.w_gu, w.w_down, 0.0, t, None, act, ye)
                                                      for _, w, _ in moe], cost, "experts", [lambda w=w: R.grouped_gated_ffn(
                                                          xs, loffs, w.w_gu, w.w_down, 7.0, t, None, act, ye) for w in like_moe], cost)
    del act, xs
    R.route_grouped(zr, model.groups(f), r)
    R.route_scatter(h, r, torch.empty(t * slots, d, dtype=BF, device=dev), f.always)
    R.route_corrected(zr, like_moe[0].correction, EXPERTS, lr)
    R.route_scatter(h, lr, torch.empty(t * slots, d, dtype=BF, device=dev))
    tab.add(ph, "routed: combine + output norm + residual + norm", [lambda l=l: W.sandwich_norm(
        x, ye, l.post2, l.norm1, h, 1e-6, d, routing=r) for _, _, l in moe], (t * slots * d * 2 + t * d * 10, 0),
        "combine + norm + residual", [lambda: R.combine_post_norm(ye, lr, one, 1e-6, d, x, h) for _ in moe],
        (t * slots * d * 2 + t * d * 10, 0))


def decode_kernels(tab: Table, model: NizoraxModel, like, b: int, ctx: int):
    cfg, d, dev = model.cfg, model.cfg.width, model.device
    attn_ls, light, dense, moe = kinds(model)
    cache = filled_cache(model, b, ctx, 32)
    eng = model.make_decode_engine(cache, b)
    eng.bind(list(range(b)), [1] * b)
    eng.reserve(4)
    if not (eng.fused and b <= eng.matvec_rows):
        return
    c, ph, each = eng._context(b), f"decode b{b} ctx {ctx}", list(enumerate(model.w.layers))
    rnd = lambda *s, dtype=F32: torch.randn(*s, device=dev, dtype=dtype)                     # noqa: E731
    x, x2, y, h = rnd(b, d), rnd(b, d), rnd(b, d), rnd(b, d)
    ls = list(enumerate(like.w.layers))
    like_moe, like_dense = ([l for _, l in ls if isinstance(l.mlp, k)] for k in (RoutedFfWeights, DenseFfWeights))
    like_rec = [(i, l.mix) for i, l in ls if isinstance(l.mix, rodapel.WkvWeights)]
    like_win = [(i, l.mix) for i, l in ls if isinstance(l.mix, rodapel.WindowWeights)]
    lcache = filled_cache(like, b, ctx, 32)
    leng = like.make_decode_engine(lcache, b)
    leng.bind(list(range(b)), [1] * b)
    leng.reserve(4)
    lc = leng._context(b)
    pend = N.Pending(y, like.w.layers[0].norm1)
    tab.add(ph, "output norm + residual + norm + convolution", [lambda i=i, l=l: W.sandwich_step(
        x, y, l.post1, l.norm2, h, 1e-6, d, (l.conv1, cache.layer_state(i, "conv1"), c.slots), pdl=True) for i, l in each],
        (b * d * 4 * (2 * TAPS + 3) + d * 4 * (TAPS + 4), 0), "output norm + residual",
        [lambda l=l: N.post_norm_add(y, l.norm1, 1e-6, d, x, None, pdl=True) for _, l in ls], (b * d * 12 + d * 4, 0))
    # projections of finished rows
    w0, l0 = attn_ls[0][1], like_win[0][1]
    raw, lraw = rnd(b, w0.w_in.n), rnd(b, l0.w_in.n)
    tab.add(ph, "attention: input projection", [lambda w=w: N.rows_in(h, w.w_in.w, raw, pdl=True) for _, w, _ in attn_ls],
            (w0.w_in.n * d * 2, 0), "output norm + projection",
            [lambda w=w: N.postnorm_in(x, pend, 1e-6, d, x2, w.w_in.w, lraw, pdl=True) for _, w in like_win], (l0.w_in.n * d * 2, 0))
    m = w0.spec
    out = rnd(b, m.heads, m.vdim, dtype=BF)
    scr = model.scratch(2 * m.heads, m.kv_heads, m.vdim, b, model.attention_splits(m, b, c.max_len, m.window))
    lscr = like.scratch(m.heads, m.kv_heads, HD, b, like.attention_splits(l0.spec, b, lc.max_len, WINDOW))
    kv = b * WINDOW * 2 * m.kv_heads * HD * 2
    tab.add(ph, "attention: rotation + append + two maps", [lambda i=i, w=w: P.flash_decode_scored(
        cache.k[i], cache.v[i], c.block_table, c.positions, w.mods, out, scr, m.heads, m.dim, m.vdim, raw=raw, n_rows=b,
        window=WINDOW, head_norm=True, normed=False, inv_freq=w.inv_freq, neighbours=True, diff=w.diff, pdl=True)
        for i, w, _ in attn_ls], (kv, 0), "head norms + append + attention, same window", [lambda i=i, w=w: P.flash_decode_scored(
            lcache.k[i], lcache.v[i], lc.block_table, lc.positions, w.mods, out, lscr, m.heads, HD, HD, raw=lraw, q_w=w.q_norm,
            k_w=w.k_norm, eps=1e-6, n_rows=b, window=WINDOW, head_norm=True, gate_col=w.gate_at, pdl=True) for i, w in like_win])
    # lightning
    g0, r0 = light[0][1], like_rec[0][1]
    s = g0.spec
    _, at_k, at_v, at_g = g0.at
    raw, o, a = rnd(b, g0.w_in.n), rnd(b, g0.w_o.k), rnd(b, g0.w_o.k, dtype=BF)
    wraw, wout = rnd(b, r0.w_in.n), rnd(b, r0.inner_p, dtype=BF)
    tab.add(ph, "lightning: state", [lambda i=i, w=w: W.lightning_step(raw, at_k, at_v, w.decay, c.slots, cache.layer_state(i, "state"),
                                                                       o, pdl=True) for i, w, _ in light],
            (b * s.heads * s.dim * s.vdim * 8, 0), "WKV step", [lambda i=i, w=w: wkv.wkv_decode(
                wraw, w.inner_p, w.w2, w.w0, w.u, w.norm, 1e-6, lc.slots, lcache.layer_state(i, "wkv"), lcache.layer_state(i, "prev"),
                x, wout, pdl=True) for i, w in like_rec], (r0.w2.numel() * 2 + b * r0.spec.heads * r0.spec.dim ** 2 * 8, 0))
    tab.add(ph, "lightning: norm + gate + output projection", [lambda w=w: W.gated_out(o, raw[:, at_g:], w.norm, 1e-6, w.w_o.w, y, pdl=True)
                                                               for _, w, _ in light], (d * g0.w_o.k * 2, 0),
            "output projection", [lambda w=w: N.matvec_out(a, w.w_o.w, y, pdl=True) for _, w, _ in light])
    # dense
    f = dense[0][1]
    ff, lff = f.w_up.n, like_dense[0].mlp.w_down.k
    z, act = rnd(b, ff), rnd(b, lff, dtype=BF)
    tab.add(ph, "dense: up projection", [lambda w=w: N.rows_in(h, w.w_up.w, z, pdl=True) for _, w, _ in dense], (ff * d * 2, 0),
            "output norm + gate/up", [lambda l=l: N.postnorm_gated(x, pend, 1e-6, d, x2, l.mlp.w_gu.w, 7.0, act, pdl=True)
                                      for l in like_dense], (2 * lff * d * 2, 0))
    tab.add(ph, "dense: activation + down projection", [lambda w=w: W.poly_out(z, w.act, 1e-6, w.spec.ff, w.w_down.w, y, pdl=True)
                                                        for _, w, _ in dense], (ff * d * 2, 0), "down",
            [lambda l=l: N.matvec_out(act, l.mlp.w_down.w, y, pdl=True) for l in like_dense], (lff * d * 2, 0))
    # routed
    f = moe[0][1]
    slots, ex = TOP + f.always, f.w_down.k
    r, lr = model.routing(f, c), like.routing(like_moe[0].mlp, lc)
    zr, lz = rnd(b, EXPERTS), rnd(b, like_moe[0].mlp.router.shape[0])
    tab.add(ph, "routed: router + choice", [lambda w=w: R.grouped_router(h, w.router, model.groups(w), zr, eng.ticket, r, pdl=True)
                                            for _, w, _ in moe], (EXPERTS * d * 2, 0), "output norm + router + choice",
            [lambda l=l: R.postnorm_router(x, pend, 1e-6, d, x2, l.mlp.router, l.mlp.correction, EXPERTS, lz, leng.ticket, lr, pdl=True)
             for l in like_moe], (EXPERTS * d * 2, 0))
    for i in range(b):                     # fixed, distinct experts: every slot has work
        pick = torch.arange(i * slots, (i + 1) * slots, dtype=torch.int32) % EXPERTS
        r.idx[i], lr.idx[i] = pick, pick
    r.weights.fill_(0.25)
    lr.weights.fill_(0.25)
    acte = rnd(b * slots, ex, dtype=BF)
    tab.add(ph, "routed: experts' gate/up", [lambda w=w: R.postnorm_expert(h, w.w_gu.w, 0.0, r, acte, pdl=True) for _, w, _ in moe],
            (b * slots * 2 * ex * d * 2, 0), "the same kernel", [lambda l=l: R.postnorm_expert(x, l.mlp.w_gu.w, 7.0, lr, acte, pdl=True)
                                                                 for l in like_moe])
    tab.add(ph, "routed: experts' down", [lambda w=w: R.expert_out(acte, w.w_down.w, r, h, y, pdl=True) for _, w, _ in moe],
            (b * slots * ex * d * 2, 0), "the same kernel", [lambda l=l: R.expert_out(acte, l.mlp.w_down.w, lr, x, y, pdl=True)
                                                             for l in like_moe])


def main(argv=None) -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--sizes", default="2048,4096")
    ap.add_argument("--layers", type=int, default=8)
    ap.add_argument("--tokens", default="2048,8192")
    ap.add_argument("--batches", default="1,8,64")
    ap.add_argument("--ctx", type=int, default=4608)
    ap.add_argument("--kernels", action="store_true", help="also the new kernels against their rooflines")
    a = ap.parse_args(argv)
    tokens, batches = [int(x) for x in a.tokens.split(",")], [int(x) for x in a.batches.split(",")]
    dev = torch.device("cuda:0")
    for width in (int(x) for x in a.sizes.split(",")):
        cfg, lcfg = nizorax_cfg(width, a.layers), like_cfg(width, a.layers)
        model = NizoraxModel(build_weights(cfg, random_tensors(cfg, 0, dev), dev))
        ours = run_models(model, tokens, batches, a.ctx)
        like = rodapel.RodapelModel(rodapel.build_weights(lcfg, rodapel.random_tensors(lcfg, 0, dev), dev))
        theirs = run_models(like, tokens, batches, a.ctx)
        print(json.dumps({"width": width, "layers": a.layers, "ctx": a.ctx, "unit": "tokens/s", "nizorax": ours, "rodapel": theirs,
                          "weight_bytes": [model.w.nbytes(), like.w.nbytes()],
                          "ratio": {k: round(ours[k] / theirs[k], 3) for k in ours if ours[k] and theirs[k]}}), flush=True)
        if a.kernels:
            with torch.no_grad():
                for b in batches:
                    decode_kernels(Table(width), model, like, b, a.ctx)
                    torch.cuda.empty_cache()
                for t in tokens:
                    prefill_kernels(Table(width), model, like, t)
                    torch.cuda.empty_cache()
            GemmStatus.check(dev)
        del model, like
        torch.cuda.empty_cache()
    return 0


if __name__ == "__main__":
    sys.exit(main())
