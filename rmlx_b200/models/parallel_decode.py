"""Cached decode of parallel-block models: three launches per layer, one CUDA graph per step.

  1. norm + merged [q; k; v; up] projection (+ xIELU)          (parallel_in)
  2. query / key norm + KV append + paged split-KV attention   (flash_decode_scored, fused form)
  3. output + down projections, layer scales, residual sum     (parallel_out)

Batches beyond ``MATVEC_ROWS`` rows, head sizes outside the fused attention kernel and 32-bit models
run the five-launch block of the prompt path instead (GEMMs with one row per sequence), captured the
same way."""
from __future__ import annotations

from typing import Optional

import torch

from .. import _lib
from ..ops import parallel_block as P
from ..ops.parallel_block import pad8
from .decode_engine import DecodeEngineBase
from .posudra import BlockBuffers, PosudraModel

# Above this many rows the GEMM form of the step is faster (measured, us per layer at 4096 cached tokens,
# mat-vec against GEMM: width 2048: 2 rows 76 / 141, 4 rows 137 / 151, 8 rows 215 / 153; width 4096: 2 rows
# 169 / 266, 4 rows 286 / 239, 8 rows 522 / 258).
MATVEC_ROWS = 3


class ParallelBlockDecode(DecodeEngineBase):
    def __init__(self, model: PosudraModel, cache, max_batch: int = 1, use_graph: bool = True, pdl: bool = True,
                 greedy: bool = True, matvec_rows: int = MATVEC_ROWS):
        super().__init__(model, cache, max_batch, use_graph, pdl, greedy)
        self.bufs = BlockBuffers(model, max_batch, raw_f32=True)
        self.matvec_rows = matvec_rows
        self.max_len = cache.max_blocks_per_seq * cache.block_size
        # every layer fits the three-launch form: bf16, head sizes of the fused attention kernel, and
        # at least one row's activations in a block's shared memory
        self.fused = all(
            model.tensor_core_decode(lw) and P.gemv_max_rows(model.width_p) > 0 and
            P.gemv_max_rows(lw.spec.mixer.heads * pad8(lw.spec.mixer.vdim) + lw.ff) > 0 for lw in model.w.layers)
        self._plan = {}
        for nb in self.buckets:       # planned up front: a step that allocates nothing can be recorded natively
            self._scratch(nb)

    def _scratch(self, nb: int):
        """Per layer, the split-KV scratch of a step of ``nb`` rows (None: attention_any)."""
        if nb not in self._plan:
            m = self.model
            self._plan[nb] = [m.scratch(lw, nb, m.decode_splits(lw, nb, self.max_len))
                              if m.tensor_core_decode(lw) else None for lw in m.w.layers]
        return self._plan[nb]

    def _run_step(self, nb: Optional[int] = None) -> None:
        m, cfg, w, pdl, cache = self.model, self.cfg, self.model.w, self.pdl, self.cache
        nb = self.B if nb is None else nb
        n0 = _lib.launch_count()
        scratch = self._scratch(nb)
        positions, table, x = self.positions[:nb], self.block_table[:nb], self.bufs.x[:nb]
        P.embed_scaled(w.embed, self.tokens[:nb], cfg.embedding_scale, x, pdl=False)
        fused = self.fused and nb <= self.matvec_rows
        for li, lw in enumerate(w.layers):
            mx, k, v = lw.spec.mixer, cache.k[li], cache.v[li]
            if fused:
                _, act, _, attn = self.bufs.layer(lw, nb)
                raw = self.bufs.raw32(lw, nb)
                P.norm_in_proj(x, lw.norm1, cfg.norm_eps, cfg.width, lw.w_in.w, lw.n_raw, lw.act_p, lw.act_n, raw, act,
                               pdl=pdl)
                P.flash_decode_scored(k, v, table, positions, lw.mods, attn, scratch[li], mx.heads, mx.dim, mx.vdim,
                                      raw=raw, q_w=lw.q_norm, k_w=lw.k_norm, eps=cfg.norm_eps, n_rows=nb, pdl=pdl)
                P.gemv_out_add(attn.view(nb, -1), lw.w_o.w, lw.ls1, act, None if lw.w_down is None else lw.w_down.w,
                               lw.ls2, x, pdl=pdl)
                continue

            def attend(lw, q, attn, li=li, mx=mx, k=k, v=v):
                if scratch[li] is None:
                    P.attention_any(q, k, v, table, positions, None, lw.mods, attn, pdl=pdl)
                else:
                    P.flash_decode_scored(k, v, table, positions, lw.mods, attn, scratch[li], mx.heads, mx.dim,
                                          mx.vdim, q=q, n_rows=nb, pdl=pdl)

            m.block(li, self.bufs, nb, cache, table, positions, None, attend, pdl=pdl)
        m.logits(x, self.bufs.h[:nb], out=self.logits[:nb], pdl=pdl)
        self._finish_step(pdl=pdl and m.dtype == torch.bfloat16, n0=n0, nb=nb)
