#!/usr/bin/env python
"""Prefill and decode throughput of the parallel-block decoder (Posudra) beside the framework's dense
decoder at equal size, and every kernel of both against its roofline. Random weights, one GPU, bf16.

    python benchmarks/bench_parallel_block.py [--sizes 2048,4096,8192] [--layers 8] [--kernels]
    python bench.py --suite parallel_block ...       # the same

Equal size: same width, heads and head size, the same number of parameters per layer (a gated
feed-forward of inner width I has three matrices, the xIELU one two, so ff = 3 I / 2), no vocabulary
effect (both LM heads are 32768 rows). Prefill: one prompt of ``--tokens``; decode: B sequences of
``--ctx`` cached tokens, one captured step per token. Timing: CUDA events after warm-up, the layers'
weights together exceed L2, so nothing is reused between steps. Kernel times: graph-captured
loops over all layers (each with its own weights and pages), after a pause in which the clocks recover
from the power cap. "roofline" is the larger of bytes / copy
bandwidth and FLOPs / burst GEMM rate of MEASURED_PEAKS.json."""
from __future__ import annotations

import argparse
import json
import os
import sys
import time

import torch

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
from rmlx_b200._lib import NativeError  # noqa: E402
from rmlx_b200.config import (FeedForwardType, ParallelLayerSpec, PosudraConfig, ScoredAttentionSpec,  # noqa: E402
                              TransformerConfig)
from rmlx_b200.models.posudra import PosudraModel, build_weights, random_tensors  # noqa: E402
from rmlx_b200.models.ragged import Entry, RaggedBatch  # noqa: E402
from rmlx_b200.models.transformer import TransformerModel  # noqa: E402
from rmlx_b200.models.weights import random_on_device  # noqa: E402
from rmlx_b200.ops import decode as D  # noqa: E402
from rmlx_b200.ops import parallel_block as P  # noqa: E402
from rmlx_b200.ops.gemm import GemmStatus  # noqa: E402

# width: (query heads, kv heads, gated inner width)
SIZES = {2048: (16, 4, 8192), 4096: (32, 8, 14336), 8192: (64, 8, 28672)}
HD, VOCAB = 128, 32768


def peaks():
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "MEASURED_PEAKS.json")
    if os.path.exists(path):
        with open(path) as f:
            p = json.load(f)
        return p["hbm_gbs"] * 1e9, p["bf16_tflops"] * 1e12
    return 6.65e12, 1.59e15


def posudra_cfg(width: int, layers: int) -> PosudraConfig:
    hq, hkv, inter = SIZES[width]
    spec = ParallelLayerSpec(ScoredAttentionSpec(hq, hkv, HD, HD, HD ** -0.5, 50.0), inter * 3 // 2)
    return PosudraConfig(VOCAB, width, [spec] * layers, 1e-6, 1.0).validate()


def dense_cfg(width: int, layers: int, max_len: int) -> TransformerConfig:
    hq, hkv, inter = SIZES[width]
    return TransformerConfig(hidden_size=width, num_heads=hq, num_kv_heads=hkv, head_dim=HD, num_layers=layers,
                             vocab_size=VOCAB, max_seq_len=max_len, ff_type=FeedForwardType.gated(inter),
                             name="dense").validate()


def ev_ms(fn, iters: int, warmup: int = 3) -> float:
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(iters):
        fn()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / iters


def graph_us(fn, launches: int, iters: int = 10) -> float:
    """Microseconds per launch of ``fn`` (a loop of ``launches`` launches), captured and replayed."""
    fn()
    torch.cuda.synchronize()
    time.sleep(0.3)          # the GEMM loops before may have pushed the part into its power cap
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        fn()
    warm = max(3, int(20.0 / max(ev_ms(g.replay, 1, 1), 0.02)))          # ~20 ms: clocks settle
    return ev_ms(g.replay, max(iters, warm // 2), warm) * 1e3 / launches


def filled_cache(model, batch: int, ctx: int, extra: int):
    bps = (ctx + extra + 15) // 16
    cache = model.new_cache(1 + batch * bps, max_seqs=batch, max_blocks_per_seq=bps)
    for s in range(batch):
        cache.add_sequence(s)
        cache.reserve(s, ctx)
        cache.commit(s, ctx)
    for k, v in zip(cache.k, cache.v):
        k.normal_(0, 1)
        v.normal_(0, 1)
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
    def __init__(self):
        self.rows, (self.bw, self.fl) = [], peaks()

    def add(self, model, phase, kernel, us, nbytes, flops):
        floor = max(nbytes / self.bw, flops / self.fl) * 1e6
        self.rows.append({"model": model, "phase": phase, "kernel": kernel, "us": round(us, 2),
                          "roofline_us": round(floor, 2), "frac": round(floor / us, 3)})


def posudra_kernels(tab: Table, model: PosudraModel, tokens, batches, ctx):
    cfg, w, n = model.cfg, model.w, len(model.w.layers)
    spec = cfg.layers[0]
    m, d, ff = spec.mixer, cfg.width, spec.ff
    nq, nk, nv = m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim
    nin, no = nq + nk + nv + ff, m.heads * m.vdim
    from rmlx_b200.models.posudra import BlockBuffers
    for t in tokens:
        cache = model.new_cache(t // 16 + 2, max_seqs=1, max_blocks_per_seq=t // 16 + 1)
        cache.add_sequence(0)
        batch = RaggedBatch.plan([Entry(0, [1] * t)], cache, m.heads)
        cache.reserve(0, t)
        batch.upload(model.device)
        bufs = BlockBuffers(model, t)
        bufs.x.normal_()
        views = [bufs.layer(w.layers[0], t)]        # the layers are alike: one set of activations
        for v in views[0]:
            v.normal_()
        for k, v in zip(cache.k, cache.v):
            k.normal_()
            v.normal_()
        loops = {
            "norm": lambda: [P.rms_norm_f32(bufs.x, lw.norm1, 1e-6, bufs.h, d) for lw in w.layers],
            "in projection + xIELU": lambda: [P.in_proj(bufs.h, lw.w_in.w, lw.n_raw, lw.act_p, lw.act_n, *views[0][:2])
                                              for lw in w.layers],
            "qk norm + append": lambda: [P.qk_norm_append(views[0][0], lw.q_norm, lw.k_norm, 1e-6, views[0][2], cache.k[i],
                                                          cache.v[i], cache.block_table, batch.positions, batch.token_seq,
                                                          m.heads, m.dim, m.vdim) for i, lw in enumerate(w.layers)],
            "attention": lambda: [P.flash_prefill_scored(views[0][2], cache.k[i], cache.v[i], cache.block_table,
                                                         batch.tiles, lw.mods, views[0][3], lanes=batch.lanes) for i, lw in enumerate(w.layers)],
            "out projections + residual": lambda: [P.out_proj_add(views[0][3].view(t, -1), lw.w_o.w, lw.ls1, views[0][1],
                                                                  lw.w_down.w, lw.ls2, bufs.x) for lw in w.layers]}
        cost = {"norm": (t * d * 6, 0), "in projection + xIELU": (nin * d * 2 + t * (d + nin) * 2, 2.0 * t * d * nin),
                "qk norm + append": (t * (nq + nk + nv) * 4, 0),
                "attention": (t * (2 * no + nk + nv) * 2, 2.0 * m.heads * (m.dim + m.vdim) * t * (t + 1) / 2),
                "out projections + residual": ((no + ff) * d * 2 + t * (no + ff) * 2 + t * d * 8, 2.0 * t * d * (no + ff))}
        for name, fn in loops.items():
            tab.add("posudra", f"prefill {t}", name, graph_us(fn, n), *cost[name])
        del cache, bufs, views
    for b in batches:
        cache = filled_cache(model, b, ctx, 32)
        eng = model.make_decode_engine(cache, b)
        eng.bind(list(range(b)), [1] * b)
        eng.reserve(4)
        bufs, pos, table = eng.bufs, eng.positions, eng.block_table
        bufs.x.normal_()
        scr = eng._scratch(b)
        lw0 = w.layers[0]
        raw16, act, q, attn = bufs.layer(lw0, b)
        raw = bufs.raw32(lw0, b)
        kv = b * ctx * (nk + nv) * 2
        if eng.fused and b <= eng.matvec_rows:
            loops = {
                "norm + in projection + xIELU": lambda: [P.norm_in_proj(bufs.x, lw.norm1, 1e-6, d, lw.w_in.w, lw.n_raw,
                                                                        lw.act_p, lw.act_n, raw, act, pdl=True) for lw in w.layers],
                "qk norm + append + attention": lambda: [P.flash_decode_scored(
                    cache.k[i], cache.v[i], table, pos, lw.mods, attn, scr[i], m.heads, m.dim, m.vdim, raw=raw,
                    q_w=lw.q_norm, k_w=lw.k_norm, eps=1e-6, n_rows=b, pdl=True) for i, lw in enumerate(w.layers)],
                "out projections + residual": lambda: [P.gemv_out_add(attn.view(b, -1), lw.w_o.w, lw.ls1, act, lw.w_down.w,
                                                                      lw.ls2, bufs.x, pdl=True) for lw in w.layers]}
        else:
            loops = {
                "norm": lambda: [P.rms_norm_f32(bufs.x, lw.norm1, 1e-6, bufs.h, d, pdl=True) for lw in w.layers],
                "in projection + xIELU": lambda: [P.in_proj(bufs.h, lw.w_in.w, lw.n_raw, lw.act_p, lw.act_n, raw16, act,
                                                            pdl=True) for lw in w.layers],
                "qk norm + append": lambda: [P.qk_norm_append(raw16, lw.q_norm, lw.k_norm, 1e-6, q, cache.k[i], cache.v[i],
                                                              table, pos, None, m.heads, m.dim, m.vdim, pdl=True)
                                             for i, lw in enumerate(w.layers)],
                "attention": lambda: [P.flash_decode_scored(cache.k[i], cache.v[i], table, pos, lw.mods, attn, scr[i],
                                                            m.heads, m.dim, m.vdim, q=q, n_rows=b, pdl=True)
                                      for i, lw in enumerate(w.layers)],
                "out projections + residual": lambda: [P.out_proj_add(attn.view(b, -1), lw.w_o.w, lw.ls1, act, lw.w_down.w,
                                                                      lw.ls2, bufs.x, pdl=True) for lw in w.layers]}
        for name, fn in loops.items():
            nb = {"norm": b * d * 6, "qk norm + append": b * (nq + nk + nv) * 4}.get(name)
            if nb is None:
                nb = kv if "attention" in name else nin * d * 2 if "in proj" in name else (no + ff) * d * 2
            tab.add("posudra", f"decode b{b} ctx {ctx}", name, graph_us(fn, n), nb, 0)
        del eng, cache
        torch.cuda.empty_cache()


def dense_kernels(tab: Table, model: TransformerModel, tokens, batches, ctx):
    from rmlx_b200.models.decode_engine import CachedDecode
    from rmlx_b200.models.prefill import _gate_up_act, _mm
    from rmlx_b200.ops.attention import flash_prefill_paged
    cfg, w, n = model.cfg, model.w, model.cfg.num_layers
    d, inter, hq, hkv = cfg.hidden_size, cfg.ff_type.intermediate_dim, model.hq, model.hkv
    nqkv, no = (hq + 2 * hkv) * HD, hq * HD
    bf = dict(dtype=torch.bfloat16, device=model.device)
    for t in tokens:
        cache = model.new_cache(t // 16 + 2, max_seqs=1, max_blocks_per_seq=t // 16 + 1)
        cache.add_sequence(0)
        cache.reserve(0, t)
        row = cache.block_table[0]
        h, qkv = torch.randn(t, d, **bf), torch.randn(t, nqkv, **bf)
        q, attn, act = torch.randn(t, hq, HD, **bf), torch.randn(t, no, **bf), torch.randn(t, inter, **bf)
        for k, v in zip(cache.k, cache.v):
            k.normal_()
            v.normal_()
        pos = torch.arange(t, dtype=torch.int32, device=model.device)
        seq = torch.zeros(t, dtype=torch.int32, device=model.device)
        loops = {
            "norm": lambda: [D.rms_norm(h, lw.norm1, 1e-6) for lw in w.layers],
            "qkv projection": lambda: [_mm(h, lw.wqkv) for lw in w.layers],
            "rope + append": lambda: [D.rope_kv_write(qkv, q, cache.k[i], cache.v[i], row.view(1, -1), pos, model.cos,
                                                      model.sin, hq, hkv, token_seq=seq) for i in range(n)],
            "attention": lambda: [flash_prefill_paged(q, cache.k[i], cache.v[i], row, 0, model.scale) for i in range(n)],
            "o projection + residual": lambda: [_mm(attn, lw.wo, residual=h) for lw in w.layers],
            "gate/up + SwiGLU": lambda: [_gate_up_act(h, lw.w_gate_up) for lw in w.layers],
            "down + residual": lambda: [_mm(act, lw.w_down, residual=h) for lw in w.layers]}
        cost = {"norm": (t * d * 4, 0), "qkv projection": (nqkv * d * 2 + t * (d + nqkv) * 2, 2.0 * t * d * nqkv),
                "rope + append": (t * nqkv * 4, 0),
                "attention": (t * (2 * no + 2 * hkv * HD) * 2, 4.0 * hq * HD * t * (t + 1) / 2),
                "o projection + residual": (no * d * 2 + t * (no + 2 * d) * 2, 2.0 * t * d * no),
                "gate/up + SwiGLU": (2 * inter * d * 2 + t * (d + inter) * 2, 4.0 * t * d * inter),
                "down + residual": (inter * d * 2 + t * (inter + 2 * d) * 2, 2.0 * t * d * inter)}
        for name, fn in loops.items():
            tab.add("dense", f"prefill {t}", name, graph_us(fn, n), *cost[name])
        del cache
    for b in batches:
        cache = filled_cache(model, b, ctx, 32)
        eng = model.make_decode_engine(cache, b)
        eng.bind(list(range(b)), [1] * b)
        eng.reserve(4)
        kv = b * ctx * 2 * hkv * HD * 2
        h, h2 = torch.randn(b, d, **bf), torch.randn(b, d, **bf)
        if isinstance(eng, CachedDecode):
            splits, scr = eng._fd_plan(b)
            attn = eng.attn.view(b, -1)
            act = eng.dense_act[:b]
            loops = {
                "norm + qkv + rope + append": lambda: [D.rms_qkv_rope(h, lw.wqkv, lw.norm1, 1e-6, eng.q, cache.k[i], cache.v[i],
                                                                      eng.block_table, eng.positions, model.cos, model.sin, hq,
                                                                      hkv, pdl=True) for i, lw in enumerate(w.layers)],
                "attention": lambda: [D.flash_decode_paged(eng.q, cache.k[i], cache.v[i], eng.block_table, eng.seq_lens,
                                                           model.scale, splits, scr, 0, out=eng.attn, pdl=True) for i in range(n)],
                "o projection + residual": lambda: [D.rms_gemv(attn, lw.wo, None, 1e-6, residual=h, out=h2, pdl=True)
                                                    for lw in w.layers],
                "norm + gate/up + SwiGLU": lambda: [D.rms_gate_up_swiglu(h2, lw.w_gate_up, lw.norm2, 1e-6, out=act, pdl=True)
                                                    for lw in w.layers],
                "down + residual": lambda: [D.rms_gemv(act, lw.w_down, None, 1e-6, residual=h2, out=h, pdl=True)
                                            for lw in w.layers]}
        else:
            splits, scr = eng._fd_plan(b)
            attn, act = torch.randn(b, no, **bf), torch.randn(b, inter, **bf)
            qkv = torch.randn(b, nqkv, **bf)
            loops = {
                "norm": lambda: [D.rms_norm(h, lw.norm1, 1e-6) for lw in w.layers],
                "qkv projection": lambda: [_mm(h, lw.wqkv) for lw in w.layers],
                "rope + append": lambda: [D.rope_kv_write(qkv, eng.q, cache.k[i], cache.v[i], eng.table, eng.positions,
                                                          model.cos, model.sin, hq, hkv, token_seq=eng.rows) for i in range(n)],
                "attention": lambda: [D.flash_decode_paged(eng.q, cache.k[i], cache.v[i], eng.table, eng.seq_lens, model.scale,
                                                           splits, scr, 0) for i in range(n)],
                "o projection + residual": lambda: [_mm(attn, lw.wo, residual=h) for lw in w.layers],
                "gate/up + SwiGLU": lambda: [_gate_up_act(h, lw.w_gate_up) for lw in w.layers],
                "down + residual": lambda: [_mm(act, lw.w_down, residual=h) for lw in w.layers]}
        for name, fn in loops.items():
            if name == "down + residual" and isinstance(eng, CachedDecode) and min(b, 4) * inter * 4 > 220 * 1024:
                continue                 # its activations do not fit the mat-vec's shared memory
            nb = kv if name == "attention" else b * d * 4 if name == "norm" else b * nqkv * 4 if name == "rope + append" \
                else nqkv * d * 2 if "qkv" in name else no * d * 2 if "o proj" in name else \
                2 * inter * d * 2 if "gate" in name else inter * d * 2
            tab.add("dense", f"decode b{b} ctx {ctx}", name, graph_us(fn, n), nb, 0)
        del eng, cache
        torch.cuda.empty_cache()


def main(argv=None) -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--sizes", default="2048,4096,8192")
    ap.add_argument("--layers", type=int, default=8)
    ap.add_argument("--tokens", default="2048,8192")
    ap.add_argument("--batches", default="1,8,64")
    ap.add_argument("--ctx", type=int, default=4096)
    ap.add_argument("--kernels", action="store_true", help="also every kernel against its roofline")
    a = ap.parse_args(argv)
    tokens, batches = [int(x) for x in a.tokens.split(",")], [int(x) for x in a.batches.split(",")]
    dev = torch.device("cuda:0")
    for width in (int(x) for x in a.sizes.split(",")):
        tab = Table()
        cfg = posudra_cfg(width, a.layers)
        model = PosudraModel(build_weights(cfg, random_tensors(cfg, 0, dev), dev))
        ours = run_models(model, tokens, batches, a.ctx)
        if a.kernels:
            posudra_kernels(tab, model, tokens, batches, a.ctx)
        nbytes = model.w.nbytes()
        del model
        torch.cuda.empty_cache()
        max_len = max(max(tokens), a.ctx + 128)
        model = TransformerModel(random_on_device(dense_cfg(width, a.layers, max_len), dev, None))
        dense = run_models(model, tokens, batches, a.ctx)
        if a.kernels:
            dense_kernels(tab, model, tokens, batches, a.ctx)
        print(json.dumps({"width": width, "heads": SIZES[width][:2], "layers": a.layers, "ctx": a.ctx, "unit": "tokens/s",
                          "posudra": ours, "dense": dense, "weight_bytes": [nbytes, model.w.nbytes()],
                          "ratio": {k: round(ours[k] / dense[k], 3) for k in ours if ours[k] and dense[k]}}), flush=True)
        for r in tab.rows:
            print(json.dumps({"width": width, **r}), flush=True)
        del model
        torch.cuda.empty_cache()
    return 0


if __name__ == "__main__":
    sys.exit(main())
