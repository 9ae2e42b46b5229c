#!/usr/bin/env python
"""Prefill and decode throughput of the twin-norm decoder (Nugosun) beside the framework's closest model, the post-norm
decoder (Rodapel), at equal size, and its new kernels beside the like kernels of the framework's other models, each
against its roofline. Random weights, one GPU, bf16.

    python benchmarks/bench_twin_norm.py [--sizes 2048,4096] [--layers 8] [--kernels]
    python bench.py --suite twin_norm ...       # the same

Layers come in fours: latent attention + dense, gated linear attention + routed, chunked attention beside state-space
heads + routed, latent attention on the first one's rows + routed. Equal size: the post-norm decoder has the same
width, attention heads (size 128), latent widths, expert count and widths, top k, and as many dense layers; its windows
are as long as the chunks. Prefill: one prompt of ``--tokens``; decode: B sequences of ``--ctx`` cached tokens, one
captured step per token. Timing: CUDA events after warm-up; the layers' weights together exceed L2. Kernel times:
graph-captured loops over all layers of a kind (each with its own weights and pages). "roofline" is the largest of
bytes / copy bandwidth, tensor FLOPs / burst GEMM rate (MEASURED_PEAKS.json) and, for the recurrences, fp32 operations
/ (SMs x 128 a clock at the top clock)."""
from __future__ import annotations

import argparse
import json
import os
import sys
from dataclasses import replace

import torch

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
from bench_parallel_block import VOCAB  # noqa: E402
from bench_post_norm import HD, SIZES, TOP, WINDOW, EXPERTS, Table, filled_cache, rodapel_cfg, run_models  # noqa: E402

from rmlx_b200.config import (ChosenFfSpec, ChunkedAttentionSpec, GlaSpec, LatentAttentionSpec, NugosunConfig, PairSpec,  # noqa: E402
                              RotarySpec, StateSpaceSpec, SwigluFfSpec, TwinNormLayerSpec)
from rmlx_b200.models import rodapel  # noqa: E402
from rmlx_b200.models.nugosun import GlaWeights, NugosunModel, PairWeights, build_weights, random_tensors  # noqa: E402
from rmlx_b200.models.ragged import Entry, RaggedBatch  # noqa: E402
from rmlx_b200.models.ragged_model import Buffers, DenseFfWeights, LatentWeights, RoutedFfWeights, StepContext  # noqa: E402
from rmlx_b200.ops import parallel_block as P  # noqa: E402
from rmlx_b200.ops import post_norm as N  # noqa: E402
from rmlx_b200.ops import routed as R  # noqa: E402
from rmlx_b200.ops import scan as S  # noqa: E402
from rmlx_b200.ops import twin_norm as TN  # noqa: E402
from rmlx_b200.ops import wkv as W  # noqa: E402
from rmlx_b200.ops.gemm import GemmStatus, gemm_bf16  # noqa: E402

BF = torch.bfloat16


def nugosun_cfg(width: int, layers: int) -> NugosunConfig:
    hq, hkv, inner, ex = SIZES[width]
    lat = LatentAttentionSpec(hq, 128, 64, 128, 512, 192 ** -0.5, q_rank=3 * width // 8)
    rot = RotarySpec(500000.0, 64, {"factor": 4.0, "original": 8192.0, "fast": 32.0, "slow": 1.0})
    pair = PairSpec(ChunkedAttentionSpec(hq, hkv, HD, HD, HD ** -0.5, rot, 50.0, WINDOW),
                    StateSpaceSpec(width // 64, 64, 128, 1, 4, 1), 1.0, 1.0)
    gla, moe = GlaSpec(width // 256, 128, 256, 16.0), ChosenFfSpec(EXPERTS, TOP, ex)
    out = []
    for i in range(0, layers, 4):
        out += [TwinNormLayerSpec(lat, SwigluFfSpec(inner)), TwinNormLayerSpec(gla, moe), TwinNormLayerSpec(pair, moe),
                TwinNormLayerSpec(replace(lat, kv_from=i), moe)]
    return NugosunConfig(VOCAB, width, out[:layers], 1e-6).validate()


def kinds(model):
    ls = list(enumerate(model.w.layers))
    pick = lambda cls, part: [(i, getattr(l, part), l) for i, l in ls if isinstance(getattr(l, part), cls)]   # noqa: E731
    return (pick(LatentWeights, "mix"), pick(GlaWeights, "mix"), pick(PairWeights, "mix"), pick(DenseFfWeights, "mlp"),
            pick(RoutedFfWeights, "mlp"))


class WkvLike:
    """The WKV recurrence at the same width: heads of 64."""

    def __init__(self, width, t, dev):
        self.h = width // 64
        rnd = lambda *s, dtype=torch.float32: torch.randn(*s, device=dev, dtype=dtype)       # noqa: E731
        self.r, self.k, self.v = (rnd(t, width, dtype=BF) for _ in range(3))
        self.decay, self.w0, self.u = rnd(t, width), rnd(width), rnd(width)
        pool = torch.zeros(2, self.h * 64 * 64 + width, device=dev)
        self.state, self.prev = pool[:, :self.h * 4096].unflatten(1, (self.h, 64, 64)), pool[:, self.h * 4096:]
        self.x, self.o = rnd(t, width), rnd(t, width)
        self.rec = torch.empty(t * self.h * W.record(64), device=dev)

    def scan(self, runs):
        W.wkv_scan(self.r, self.k, self.v, self.decay, self.w0, self.u, self.state, self.prev, self.x, self.o, self.rec, runs=runs)


def prefill_kernels(tab: Table, model: NugosunModel, t: int):
    cfg, d, dev = model.cfg, model.cfg.width, model.device
    lat, gla, pairs, dense, moe = kinds(model)
    cache = model.new_cache(t // 16 + 2, max_seqs=1, max_blocks_per_seq=t // 16 + 1)
    cache.add_sequence(0)
    batch = RaggedBatch.plan([Entry(0, [1] * t)], cache, model._min_heads, model._absorb)
    cache.reserve(0, t)
    batch.upload(dev)
    c = StepContext(t, Buffers(t, dev), cache, cache.block_table, batch.positions, batch.token_seq, batch.token_seq, batch.runs, batch)
    for pool in {id(p): p for p in cache.k + cache.v if p is not None}.values():
        pool.normal_()
    rnd = lambda *s, dtype=BF: torch.randn(*s, device=dev, dtype=dtype)                      # noqa: E731
    x, h, h2, y = rnd(t, d, dtype=torch.float32), rnd(t, d), rnd(t, d), rnd(t, d, dtype=torch.float32)
    ph, each = f"prefill {t}", model.w.layers
    gemm = lambda n, k, out=2: (n * k * 2 + t * (k * 2 + n * out), 2.0 * t * n * k)          # noqa: E731
    tab.add(ph, "two norms", [lambda l=l: TN.twin_norm(x, l.norm1, h, l.norm2, h2, 1e-6, d) for l in each], (t * d * 8, 0),
            "output norm + residual", [lambda l=l: N.post_norm_add(y, l.norm1, 1e-6, d, x, h) for l in each], (t * d * 14, 0))
    # routed
    f = moe[0][1]
    z = rnd(t, EXPERTS, dtype=torch.float32)
    r = model.routing(f, c)
    tab.add(ph, "routed: choice + offsets", [lambda: R.route_chosen(z, f.correction, r) for _ in moe], (t * (EXPERTS * 4 + TOP * 8), 0),
            "corrected choice + offsets", [lambda: R.route_corrected(z, f.correction, EXPERTS, r) for _ in moe])
    R.route_chosen(z, f.correction, r)
    R.route_scatter(h, r, torch.empty(t * TOP, d, dtype=BF, device=dev))
    ye = rnd(t * TOP, d)
    tab.add(ph, "routed: combine + residual + two norms", [lambda l=l: TN.twin_norm(x, l.norm1, h, l.norm2, h2, 1e-6, d, (ye, r))
                                                           for _, _, l in moe], (t * TOP * d * 2 + t * d * 12, 0),
            "combine + norm + residual", [lambda l=l: R.combine_post_norm(ye, r, l.norm2, 1e-6, d, x, h) for _, _, l in moe],
            (t * TOP * d * 2 + t * d * 10, 0))
    del ye
    # output projections into the residual
    w = dense[0][1]
    m = lat[0][1].spec
    act, a = rnd(t, w.w_down.k), rnd(t, m.heads * m.vdim)
    n1, n2 = a.shape[1], act.shape[1]
    tab.add(ph, "mixer + dense output into the residual", [lambda i=i, w=w, l=l: P.out_proj_add(
        a, l.mix.w_o.w, model.w.ones, act, w.w_down.w, model.w.ones, x) for i, w, l in dense],
        (d * (n1 + n2) * 2 + t * ((n1 + n2) * 2 + d * 8), 2.0 * t * d * (n1 + n2)), "down, fp32 result",
        [lambda w=w: P.logits_f32(act, w.w_down.w, y) for _, w, _ in dense], gemm(d, n2, 4))
    del act, a
    # query latent
    w0 = lat[0][1]
    raw = rnd(t, w0.w_in.n)
    cq = torch.empty(t, w0.w_uq.k, dtype=BF, device=dev)
    tab.add(ph, "latent: query norm", [lambda w=w: TN.rows_norm(raw, w.q_norm, 1e-6, m.q_rank, cq) for _, w, _ in lat],
            (t * m.q_rank * 4, 0))
    q_raw = rnd(t, w0.w_uq.n)
    tab.add(ph, "latent: query up-projection", [lambda w=w: N.linear(cq, w.w_uq.w, q_raw) for _, w, _ in lat], gemm(w0.w_uq.n, w0.w_uq.k))
    q = rnd(t, m.heads, w0.dim_p + w0.rot_p)
    tab.add(ph, "latent: rotation (+ norm + append)", [lambda i=i, w=w: N.latent_append(
        q_raw, None if w.c_norm is None else raw[:, w.down_at:], w.c_norm, 1e-6, w.inv_freq, q, None, cache.k[w.source],
        c.block_table, c.positions, c.token_seq, m.heads, m.dim, m.rot_dim, m.kv_rank, w.dim_p, w.rot_p, w.lat_p)
        for i, w, _ in lat], (t * (q_raw.shape[1] + 288) * 4, 0))
    del raw, q_raw, q, cq
    # chunked attention
    pw = pairs[0][1]
    m, s = pw.left.spec, pw.right.spec
    raw = rnd(t, pw.w_in.n)
    q, attn = rnd(t, m.heads, HD), rnd(t, m.heads, HD)
    ones = torch.ones(HD, device=dev)
    rows = (m.heads + 2 * m.kv_heads) * HD
    args = lambda i: (q, cache.k[i], cache.v[i], c.block_table, c.positions, c.token_seq, m.heads, HD, HD)   # noqa: E731
    tab.add(ph, "pair: input projection", [lambda w=w: N.linear(h, w.w_in.w, raw) for _, w, _ in pairs], gemm(pw.w_in.n, d),
            "the same GEMM", [lambda w=w: gemm_bf16(h, w.w_in.w, out=raw) for _, w, _ in pairs])
    tab.add(ph, "pair: bias + rotation + norms + append", [lambda i=i, w=w: TN.rotary_norm_append(
        raw, w.left.bias, w.left.inv_freq, w.left.grow, 1e-6, *args(i)) for i, w, _ in pairs], (t * rows * 4, 0),
        "head norms + append", [lambda i=i: N.head_norm_append(raw, ones, ones, 1e-6, *args(i)) for i, _, _ in pairs])
    seen, win = sum(p % WINDOW + 1 for p in range(t)), sum(min(p + 1, WINDOW) for p in range(t))
    cost = lambda n: (t * rows * 4, 4.0 * m.heads * HD * n)                                  # noqa: E731
    tab.add(ph, "pair: chunked attention, soft cap", [lambda i=i, w=w: P.flash_prefill_scored(
        q, cache.k[i], cache.v[i], c.block_table, batch.tiles, w.left.mods, attn, lanes=batch.lanes, chunk=WINDOW) for i, w, _ in pairs],
        cost(seen), "attention, window, soft cap", [lambda i=i, w=w: P.flash_prefill_scored(
            q, cache.k[i], cache.v[i], c.block_table, batch.tiles, w.left.mods, attn, lanes=batch.lanes, window=WINDOW)
            for i, w, _ in pairs], cost(win))
    # recurrences
    like = WkvLike(d, t, dev)
    like_cost = (t * d * 14, 0, 3.0 * t * d * 64)
    o = torch.empty(t, pw.right.w_o.k, device=dev)
    rec = torch.empty(t * s.heads * S.record(s.state, s.vdim, True, s.heads // s.groups), device=dev)
    right = raw[:, pw.left.columns:]
    st = lambda i, n: cache.layer_state(i, n)                                                # noqa: E731
    tab.add(ph, "pair: convolution + recurrence", [lambda i=i, w=w: S.ssd_scan(
        right, w.right.x_at, w.right.dt_at, w.right.conv_w, w.right.conv_b, st(i, "conv"), w.right.dt_bias, w.right.a_log,
        w.right.skip, s.groups, st(i, "ssd"), o, rec, c.slots, runs=batch.runs) for i, w, _ in pairs],
        (t * (s.channels * 2 + s.inner * 4), 0, 3.0 * t * s.heads * s.state * s.vdim), "WKV recurrence",
        [lambda: like.scan(batch.runs) for _ in pairs], like_cost)
    a = torch.empty(t, pw.right.w_o.k, dtype=BF, device=dev)
    finish = [lambda: W.wkv_finish(like.o, like.r, like.w0, 1e-6, like.h, 64, a) for _ in pairs]
    tab.add(ph, "pair: gate + grouped norm", [lambda w=w: S.gated_norm(o, right, w.right.norm, 1e-6, s.norm_groups, a, True)
                                              for _, w, _ in pairs], (t * s.inner * 8, 0), "head norm + gate", finish, (t * d * 8, 0))
    del rec, raw, right
    g0 = gla[0][1]
    m = g0.spec
    raw = rnd(t, g0.w_in.n)
    z = rnd(t, g0.qk_p, dtype=torch.float32)
    o = torch.empty(t, g0.v_p, device=dev)
    rec = torch.empty(t * m.heads * S.record(m.dim, m.vdim), device=dev)
    q, k, v, g, low = (raw[:, at:] for at in g0.at)
    tab.add(ph, "gla: input projection", [lambda w=w: N.linear(h, w.w_in.w, raw) for _, w, _ in gla], gemm(g0.w_in.n, d),
            "the same GEMM", [lambda w=w: gemm_bf16(h, w.w_in.w, out=raw) for _, w, _ in gla])
    rank = g0.w_a2.shape[1]
    tab.add(ph, "gla: decay, second factor", [lambda w=w: P.logits_f32(low[:, :rank], w.w_a2, z) for _, w, _ in gla], gemm(g0.qk_p, rank, 4))
    tab.add(ph, "gla: recurrence", [lambda i=i, w=w: S.gla_scan(q, k, v, z, w.bias, m.tau, m.dim ** -0.5, st(i, "gla"), o, rec,
                                                                runs=batch.runs) for i, w, _ in gla],
            (t * (g0.qk_p * 8 + g0.v_p * 6), 0, 3.0 * t * m.heads * m.dim * m.vdim), "WKV recurrence",
            [lambda: like.scan(batch.runs) for _ in gla], like_cost)
    tab.add(ph, "gla: head norm + gate", [lambda w=w: S.gated_norm(o, g, w.norm, 1e-6, m.heads, a[:, :g0.v_p], False) for _, w, _ in gla],
            (t * g0.v_p * 8, 0), "head norm + gate", finish[:len(gla)], (t * d * 8, 0))


def decode_kernels(tab: Table, model: NugosunModel, like, b: int, ctx: int):
    """``like``: a post-norm model of equal size."""
    cfg, d, dev = model.cfg, model.cfg.width, model.device
    lat, gla, pairs, dense, moe = kinds(model)
    cache = filled_cache(model, b, ctx, 32)
    eng = model.make_decode_engine(cache, b)
    eng.bind(list(range(b)), [1] * b)
    eng.reserve(4)
    if not (eng.fused and b <= eng.matvec_rows):
        return
    c, ph = eng._context(b), f"decode b{b} ctx {ctx}"
    f32 = torch.float32
    rnd = lambda *s, dtype=f32: torch.randn(*s, device=dev, dtype=dtype)                     # noqa: E731
    x, x2, y = rnd(b, d), rnd(b, d), rnd(b, d)
    like_dense = [l.mlp for l in like.w.layers if isinstance(l.mlp, DenseFfWeights)]
    like_moe = [l for l in like.w.layers if isinstance(l.mlp, RoutedFfWeights)]
    like_wkv = [(i, l.mix) for i, l in enumerate(like.w.layers) if isinstance(l.mix, rodapel.WkvWeights)]
    like_win = [(i, l.mix) for i, l in enumerate(like.w.layers) if isinstance(l.mix, rodapel.WindowWeights)]
    pend = N.Pending(y, like.w.layers[0].norm1)
    # inputs
    w = dense[0][1]
    act = rnd(b, w.w_down.k, dtype=BF)
    raw = rnd(b, dense[0][2].mix.w_in.n)
    bytes_in = [l.mix.w_in.n * d * 2 + w.w_gu.n * d * 2 for _, w, l in dense]
    tab.add(ph, "norms + projection + gate/up", [lambda w=w, l=l: TN.twin_in(
        x, l.norm1, 1e-6, d, l.mix.w_in.w, raw, l.norm2, w.w_gu.w, act, 0.0, pdl=True) for _, w, l in dense], (bytes_in[0], 0),
        "output norm + gate/up", [lambda w=w: N.postnorm_gated(x, pend, 1e-6, d, x2, w.w_gu.w, 7.0, act, pdl=True) for w in like_dense],
        (w.w_gu.n * d * 2, 0))
    z, h2 = rnd(b, EXPERTS), rnd(b, d)
    r = model.routing(moe[0][1], c)
    rr = {l.mix.w_in.n: rnd(b, l.mix.w_in.n) for _, _, l in moe}
    total = sum(l.mix.w_in.n + EXPERTS for _, _, l in moe) * d * 2 / len(moe)
    raw2 = {l.mix.w_in.n: rnd(b, l.mix.w_in.n) for l in like_moe}
    no_shift = [l for l in like_moe if not isinstance(l.mix, rodapel.WkvWeights)]
    tab.add(ph, "norms + projection + router + choice", [lambda w=w, l=l: TN.twin_in_router(
        x, l.norm1, 1e-6, d, l.mix.w_in.w, rr[l.mix.w_in.n], l.norm2, w.router, w.correction, z, h2, eng.ticket, r, pdl=True)
        for _, w, l in moe], (total, 0), "output norm + projection", [lambda l=l: N.postnorm_in(
            x, pend, 1e-6, d, x2, l.mix.w_in.w, raw2[l.mix.w_in.n], pdl=True) for l in no_shift],
        (sum(l.mix.w_in.n for l in no_shift) * d * 2 / len(no_shift), 0))
    # outputs
    a = rnd(b, lat[0][1].w_o.k, dtype=BF)
    tab.add(ph, "mixer + dense output into the residual", [lambda w=w, l=l: P.gemv_out_add(
        a, l.mix.w_o.w, model.w.ones, act, w.w_down.w, model.w.ones, x, pdl=True) for _, w, l in dense],
        (d * (a.shape[1] + act.shape[1]) * 2, 0), "down", [lambda w=w: N.matvec_out(act, w.w_down.w, y, pdl=True) for w in like_dense],
        (d * act.shape[1] * 2, 0))
    tab.add(ph, "mixer output into the residual", [lambda w=w: P.gemv_out_add(a, w.w_o.w, model.w.ones, None, None, None, x, pdl=True)
                                                   for _, w, _ in lat], (d * a.shape[1] * 2, 0),
            "output projection", [lambda w=w: N.matvec_out(a, w.w_o.w, y, pdl=True) for _, w in like_win], (d * a.shape[1] * 2, 0))
    # experts
    ex = moe[0][1].w_down.k
    for i in range(b):                     # fixed, distinct experts: every slot has work
        r.idx[i] = torch.arange(i * TOP, (i + 1) * TOP, dtype=torch.int32) % EXPERTS
    r.weights.fill_(0.25)
    r.identity.fill_(1.0)
    acte = rnd(b * TOP, ex, dtype=BF)
    tab.add(ph, "routed: experts' gate/up", [lambda w=w: R.postnorm_expert(h2, w.w_gu.w, 0.0, r, acte, pdl=True) for _, w, _ in moe],
            (b * TOP * 2 * ex * d * 2, 0), "the same kernel", [lambda l=l: R.postnorm_expert(x, l.mlp.w_gu.w, 7.0, r, acte, pdl=True)
                                                               for l in like_moe])
    tab.add(ph, "routed: experts' down into the residual", [lambda w=w: R.expert_out(acte, w.w_down.w, r, x, x, pdl=True)
                                                            for _, w, _ in moe], (b * TOP * ex * d * 2, 0), "the same kernel",
            [lambda l=l: R.expert_out(acte, l.mlp.w_down.w, r, x, y, pdl=True) for l in like_moe])
    # latent
    w0, m = lat[0][1], lat[0][1].spec
    lraw = {w.w_in.n: rnd(b, w.w_in.n) for _, w, _ in lat}
    q_up = rnd(b, w0.w_uq.n)
    tab.add(ph, "latent: query norm + projection", [lambda w=w: P.norm_in_proj(
        lraw[w.w_in.n][:, :w.w_uq.k], w.q_norm, 1e-6, m.q_rank, w.w_uq.w, w.w_uq.n, 0.0, 0.0, q_up, None, pdl=True) for _, w, _ in lat],
        (w0.w_uq.n * w0.w_uq.k * 2, 0), "output norm + projection", [lambda w=w: N.postnorm_in(
            x, pend, 1e-6, d, x2, w.w_in.w, raw2[w.w_in.n], pdl=True) for _, w in like_win if w.w_in.n in raw2],
        (like_win[0][1].w_in.n * d * 2, 0))
    # chunked attention, state space
    pw = pairs[0][1]
    m, s = pw.left.spec, pw.right.spec
    raw = rnd(b, pw.w_in.n)
    attn = rnd(b, m.heads, HD, dtype=BF)
    scr = model.scratch(m.heads, m.kv_heads, HD, b, model.attention_splits(m, b, c.max_len, m.chunk))
    ones = torch.ones(HD, device=dev)
    c.positions.fill_(ctx - ctx % WINDOW - 1)             # the last place of a chunk: as many keys as the window
    kv = b * WINDOW * 2 * m.kv_heads * HD * 2
    fused = lambda i, w, **kw: P.flash_decode_scored(cache.k[i], cache.v[i], c.block_table, c.positions, w.left.mods, attn, scr,   # noqa: E731
                                                     m.heads, HD, HD, raw=raw, eps=1e-6, n_rows=b, head_norm=True, pdl=True, **kw)
    tab.add(ph, "pair: bias + rotation + norms + append + attention", [lambda i=i, w=w: fused(
        i, w, chunk=WINDOW, bias=w.left.bias, inv_freq=w.left.inv_freq, grow=w.left.grow) for i, w, _ in pairs], (kv, 0),
        "head norms + append + attention, window", [lambda i=i, w=w: fused(i, w, window=WINDOW, q_w=ones, k_w=ones) for i, w, _ in pairs])
    a, yo = rnd(b, pw.right.w_o.k, dtype=BF), rnd(b, pw.right.w_o.k)
    lcache = like.new_cache(4, max_seqs=b + 1)
    wraw, wout = rnd(b, like_wkv[0][1].w_in.n), rnd(b, like_wkv[0][1].inner_p, dtype=BF)
    lw = like_wkv[0][1]
    like_fns = [lambda i=i, w=w: W.wkv_decode(wraw, w.inner_p, w.w2, w.w0, w.u, w.norm, 1e-6, c.slots, lcache.layer_state(i, "wkv"),
                                              lcache.layer_state(i, "prev"), x, wout, pdl=True) for i, w in like_wkv]
    like_cost = (lw.w2.numel() * 2 + b * lw.spec.heads * lw.spec.dim ** 2 * 8, 0)
    right = raw[:, pw.left.columns:]
    st = lambda i, n: cache.layer_state(i, n)                                                # noqa: E731
    tab.add(ph, "pair: convolution + state, gate + norm (two launches)", [lambda i=i, w=w: S.ssd_decode(
        right, w.right.x_at, w.right.dt_at, w.right.conv_w, w.right.conv_b, st(i, "conv"), w.right.dt_bias, w.right.a_log,
        w.right.skip, s.groups, c.slots, st(i, "ssd"), yo, w.right.norm, 1e-6, s.norm_groups, a, pdl=True) for i, w, _ in pairs],
        (b * s.heads * s.state * s.vdim * 8 + s.channels * s.conv * 4 * (b + 1), 0), "WKV step", like_fns, like_cost)
    g0 = gla[0][1]
    m = g0.spec
    raw, a = rnd(b, g0.w_in.n), rnd(b, g0.v_p, dtype=BF)
    tab.add(ph, "gla: decay + state + head norm + gate", [lambda i=i, w=w: S.gla_decode(
        raw, w.at, w.w_a2, w.bias, m.tau, m.dim ** -0.5, w.norm, 1e-6, c.slots, st(i, "gla"), a, pdl=True) for i, w, _ in gla],
        (g0.w_a2.numel() * 2 + b * m.heads * m.dim * m.vdim * 8, 0), "WKV step", like_fns, like_cost)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--sizes", default="2048,4096")
    ap.add_argument("--layers", type=int, default=8)
    ap.add_argument("--tokens", default="2048,8192")
    ap.add_argument("--batches", default="1,8,64")
    ap.add_argument("--ctx", type=int, default=4608, help="default: the middle of a chunk")
    ap.add_argument("--kernels", action="store_true", help="also the new kernels against their rooflines")
    a = ap.parse_args(argv)
    tokens, batches = [int(x) for x in a.tokens.split(",")], [int(x) for x in a.batches.split(",")]
    dev = torch.device("cuda:0")
    for width in (int(x) for x in a.sizes.split(",")):
        cfg, lcfg = nugosun_cfg(width, a.layers), rodapel_cfg(width, a.layers)
        model = NugosunModel(build_weights(cfg, random_tensors(cfg, 0, dev), dev))
        ours = run_models(model, tokens, batches, a.ctx)
        like = rodapel.RodapelModel(rodapel.build_weights(lcfg, rodapel.random_tensors(lcfg, 0, dev), dev))
        theirs = run_models(like, tokens, batches, a.ctx)
        print(json.dumps({"width": width, "layers": a.layers, "ctx": a.ctx, "unit": "tokens/s", "nugosun": ours, "rodapel": theirs,
                          "weight_bytes": [model.w.nbytes(), like.w.nbytes()],
                          "ratio": {k: round(ours[k] / theirs[k], 3) for k in ours if ours[k] and theirs[k]}}), flush=True)
        if a.kernels:
            with torch.no_grad():
                for b in batches:
                    decode_kernels(Table(width), model, like, b, a.ctx)
                    torch.cuda.empty_cache()
                for t in tokens:
                    prefill_kernels(Table(width), model, t)
                    torch.cuda.empty_cache()
            GemmStatus.check(dev)
        del model, like
        torch.cuda.empty_cache()
    return 0


if __name__ == "__main__":
    sys.exit(main())
