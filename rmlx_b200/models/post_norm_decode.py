"""Cached decode of post-norm decoders (``models/rodapel.py``): one row per sequence, one CUDA graph per
step. In the form of a few rows the projections are mat-vec kernels that finish the previous sublayer (its
output norm and the residual sum) while they stage their input:

  windowed attention  1. q | k | v | gate projection   2. head norms + append + split-KV attention + gate
                      3. output projection
  latent attention    1. q | latent projection   2. latent norm, rotation, append   3. queries into the latent
                      space   4. split-KV latent attention (+ merge)   5. values   6. output projection
  WKV                 1. token shift + r | k | v | g | decay projections   2. recurrence, head norm, gate
                      3. output projection
  dense feed-forward  1. gate / up with the activation   2. down projection
  routed experts      1. router and choice   2. chosen experts' gate / up   3. weighted down + identity experts"""
from __future__ import annotations

import torch

from ..ops import parallel_block as P
from ..ops import post_norm as N
from ..ops import routed as R
from ..ops import wkv as W
from .layered_decode import MATVEC_ROWS, LayeredDecode  # noqa: F401
from .ragged_model import DenseFfWeights, LatentWeights, RoutedFfWeights, StepContext
from .rodapel import WindowWeights


class PostNormDecode(LayeredDecode):
    def _fits(self, lw) -> bool:
        m, f = lw.mix, lw.mlp
        if N.max_rows(m.w_o.k) < 1:
            return False
        if isinstance(m, WindowWeights) and not self.model.tensor_core_attention(m.spec):
            return False
        if isinstance(f, DenseFfWeights):
            return N.max_rows(f.w_down.k) > 0
        return f is None or R.expert_decode_fits(f.w_down.k, f.spec.top)

    def _matvec_layers(self, c: StepContext) -> None:
        x = self.model.start(self.tokens[:c.t], self.bufs)[0]
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
                scr = m.scratch(s.heads, s.kv_heads, v.shape[3], t, m.attention_splits(s, t, c.max_len, s.window))
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
