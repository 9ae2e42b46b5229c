"""Cached decode of post-norm decoders (``models/rodapel.py``): one row per sequence, one CUDA graph per
step. Up to ``MATVEC_ROWS`` rows the projections are mat-vec kernels that finish the previous sublayer (its
output norm and the residual sum) while they stage their input:

  windowed attention  1. q | k | v | gate projection   2. head norms + append + split-KV attention + gate
                      3. output projection
  latent attention    1. q | latent projection   2. latent norm, rotation, append   3. queries into the latent
                      space   4. split-KV latent attention (+ merge)   5. values   6. output projection
  WKV                 1. token shift + r | k | v | g | decay projections   2. recurrence, head norm, gate
                      3. output projection
  dense feed-forward  1. gate / up with the activation   2. down projection
  routed experts      1. router and choice   2. chosen experts' gate / up   3. weighted down + identity experts

Larger batches, head sizes outside the fused attention kernel and 32-bit models run the layers of the
ragged batch with every row a sequence of its own, captured the same way."""
from __future__ import annotations

from typing import Optional

import torch

from .. import _lib
from ..ops import parallel_block as P
from ..ops import post_norm as N
from ..ops import routed as R
from ..ops import wkv as W
from .decode_engine import DecodeEngineBase
from .rodapel import Buffers, DenseFfWeights, LatentWeights, RodapelModel, RoutedFfWeights, StepContext, WindowWeights

# Above this many rows the GEMM form of the step runs.
MATVEC_ROWS = 3


class PostNormDecode(DecodeEngineBase):
    def __init__(self, model: RodapelModel, cache, max_batch: int = 1, use_graph: bool = True, pdl: bool = True,
                 greedy: bool = True, matvec_rows: int = MATVEC_ROWS):
        super().__init__(model, cache, max_batch, use_graph, pdl, greedy)
        self.bufs = Buffers(max_batch, model.device)
        self.matvec_rows = matvec_rows
        self.max_len = cache.max_blocks_per_seq * cache.block_size
        self._planned = set()
        self.ticket = torch.zeros(1, dtype=torch.int32, device=model.device)
        self.fused = model.dtype == torch.bfloat16 and all(self._fits(lw) for lw in model.w.layers) and \
            P.gemv_max_rows(model.width_p) > 0

    def _fits(self, lw) -> bool:
        """Whether the layer has a mat-vec form: staged rows fit shared memory, head sizes the attention kernel."""
        m, f = lw.mix, lw.mlp
        if N.max_rows(self.model.width_p) < 1 or N.max_rows(m.w_o.k) < 1:
            return False
        if isinstance(m, WindowWeights) and not self.model.tensor_core_attention(m.spec):
            return False
        if isinstance(f, DenseFfWeights):
            return N.max_rows(f.w_down.k) > 0
        return f is None or R.expert_decode_fits(f.w_down.k, f.spec.top)

    def capture(self, nb: Optional[int] = None):
        """Buffers and scratch of a bucket come with its first run: one plain run first, so that the recorded
        step allocates nothing (which the native graph store asks for)."""
        nb = self.bucket() if nb is None else nb
        if nb not in self._planned:
            self._planned.add(nb)
            restore = self._snapshot()
            self._run_step(nb)
            restore()
        return super().capture(nb)

    def _context(self, nb: int) -> StepContext:
        return StepContext(nb, self.bufs, self.cache, self.block_table[:nb], self.positions[:nb], None,
                           None if self.state_slots is None else self.state_slots[:nb], None, None, self.max_len, self.pdl)

    def _run_step(self, nb: Optional[int] = None) -> None:
        m = self.model
        nb = self.B if nb is None else nb
        n0 = _lib.launch_count()
        x, h = m.embed(self.tokens[:nb], self.bufs)
        c = self._context(nb)
        if self.fused and nb <= self.matvec_rows:
            self._matvec_layers(x, c)
        else:
            for li in range(len(m.w.layers)):
                m.layer(li, x, h, c)
            m.logits(x, h, out=self.logits[:nb], pdl=self.pdl)
        self._finish_step(pdl=self.pdl and m.dtype == torch.bfloat16, n0=n0, nb=nb)

    def _matvec_layers(self, x: torch.Tensor, c: StepContext) -> None:
        m, cfg, w, pdl, t = self.model, self.model.cfg, self.model.w, self.pdl, c.t
        eps, width, wp, bf, f32 = cfg.norm_eps, cfg.width, self.model.width_p, torch.bfloat16, torch.float32
        get = c.bufs.get
        other = get("x2", t, wp, dtype=f32)
        y = get("y", t, wp, dtype=f32)
        pending = N.Pending(None, None)

        def project(weight: torch.Tensor, shift=None) -> torch.Tensor:
            """The projection of the finished residual; the two residual buffers change places."""
            nonlocal x, other
            raw = get("raw32", t, weight.shape[0], dtype=f32)
            N.postnorm_in(x, pending, eps, width, other, weight, raw, shift=shift, pdl=pdl)
            x, other = other, x
            return raw

        for li, lw in enumerate(w.layers):
            mw, s = lw.mix, lw.mix.spec
            if isinstance(mw, WindowWeights):
                raw = project(mw.w_in.w)
                k, v = c.cache.k[li], c.cache.v[li]
                attn = get("attn", t, s.heads, v.shape[3], dtype=bf)
                scr = m.scratch(s.heads, s.kv_heads, v.shape[3], t, m.window_splits(s, t, c.max_len))
                P.flash_decode_scored(k, v, c.block_table, c.positions, mw.mods, attn, scr, s.heads, s.dim, s.vdim, raw=raw,
                                      q_w=mw.q_norm, k_w=mw.k_norm, eps=eps, n_rows=t, window=s.window, head_norm=True,
                                      gate_col=mw.gate_at, pdl=pdl)
                a = attn.view(t, -1)
            elif isinstance(mw, LatentWeights):
                a = m.latent_core(li, mw, project(mw.w_in.w), c).view(t, -1)
            else:
                state, prev = c.cache.layer_state(li, "wkv"), c.cache.layer_state(li, "prev")
                raw = project(mw.w_in.w, shift=(mw.mu, prev, c.slots, mw.inner_p))
                a = get("wkv_a", t, mw.inner_p, dtype=bf)
                W.wkv_decode(raw, mw.inner_p, mw.w2, mw.w0, mw.u, mw.norm, eps, c.slots, state, prev, x, a, pdl=pdl)
            N.matvec_out(a, mw.w_o.w, y, pdl=pdl)
            pending = N.Pending(y, lw.norm1)
            f = lw.mlp
            if isinstance(f, DenseFfWeights):
                act = get("ff", t, f.w_down.k, dtype=bf)
                N.postnorm_gated(x, pending, eps, width, other, f.w_gu.w, f.spec.limit, act, pdl=pdl)
                x, other = other, x
                N.matvec_out(act, f.w_down.w, y, pdl=pdl)
                pending = N.Pending(y, lw.norm2)
            elif isinstance(f, RoutedFfWeights):
                r = m.routing(f, c)
                z = get("route_z", t, f.router.shape[0], dtype=f32)
                inner = f.w_down.k
                act = get("moe_act", t, f.spec.top, inner, dtype=bf).view(t * f.spec.top, inner)
                R.postnorm_router(x, pending, eps, width, other, f.router, f.correction, f.spec.experts, z, self.ticket, r,
                                  pdl=pdl)
                x, other = other, x
                R.postnorm_expert(x, f.w_gu.w, f.spec.limit, r, act, pdl=pdl)
                R.expert_out(act, f.w_down.w, r, x, y, pdl=pdl)
                pending = N.Pending(y, lw.norm2)
        N.post_norm_add(pending.y, pending.w, eps, width, x, None, pdl=pdl)
        P.norm_in_proj(x, w.final_norm, eps, width, w.lm_head.w, cfg.vocab_size, 0.0, 0.0, self.logits[:t], None, pdl=pdl)
