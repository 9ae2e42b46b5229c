"""Cached decode of twin-norm decoders (``models/nugosun.py``): one row per sequence, one CUDA graph per step. In the
form of a few rows one launch reads the residual for the mixer and the feed-forward, and the output projections add
to it in place:

  layer               1. norms + mixer projection beside gate / up with the activation, or the router and its choice
  latent attention    2. query norm + projection   3. rotation, latent norm, append   4. queries into the latent space
                      5. split-KV latent attention (+ merge)   6. values
  linear attention    2. decay, state, head norm, gate
  pair                2. bias, rotation, norms, append, split-KV attention   3. convolution, state   4. gate, norm
  output              mixer and dense down projection into the residual (two terms a launch)
  routed experts      chosen experts' gate / up; weighted down projections into the residual"""
from __future__ import annotations

import torch

from ..ops import parallel_block as P
from ..ops import post_norm as N
from ..ops import routed as R
from ..ops import scan as S
from ..ops import twin_norm as TN
from .layered_decode import LayeredDecode
from .nugosun import GlaWeights, PairWeights
from .ragged_model import DenseFfWeights, LatentWeights, StepContext


class TwinNormDecode(LayeredDecode):
    def _fits(self, lw) -> bool:
        m, f = lw.mix, lw.mlp
        outs = [m.left.w_o.k, m.right.w_o.k] if isinstance(m, PairWeights) else [m.w_o.k]
        if isinstance(m, PairWeights) and not self.model.tensor_core_attention(m.left.spec):
            return False
        if isinstance(m, GlaWeights) and not S.gla_decode_supported(m.spec.dim, m.spec.vdim):
            return False
        if isinstance(m, LatentWeights) and P.gemv_max_rows(m.w_uq.k) < 1:
            return False
        if isinstance(f, DenseFfWeights):
            outs.append(f.w_down.k)
        elif f is not None and not R.expert_decode_fits(f.w_down.k, f.spec.top):
            return False
        return all(P.gemv_max_rows(sum(outs[i:i + 2])) > 0 for i in range(0, len(outs), 2))

    def _mixer(self, li: int, mw, raw: torch.Tensor, c: StepContext) -> list:
        """The mixer's terms of the residual from its projection's rows."""
        m, t, pdl, eps, bf = self.model, c.t, self.pdl, self.model.cfg.norm_eps, torch.bfloat16
        get, s, ones = c.bufs.get, mw.spec, m.w.ones
        if isinstance(mw, LatentWeights):
            return [(m.latent_core(li, mw, raw, c).view(t, -1), mw.w_o, ones)]
        if isinstance(mw, GlaWeights):
            a = get("scan_a", t, mw.v_p, dtype=bf)
            S.gla_decode(raw, mw.at, mw.w_a2, mw.bias, s.tau, s.dim ** -0.5, mw.norm, eps, c.slots,
                         c.cache.layer_state(li, "gla"), a, pdl=pdl)
            return [(a, mw.w_o, ones)]
        l, r, k, v = mw.left, mw.right, c.cache.k[li], c.cache.v[li]
        attn = get("attn", t, l.spec.heads, v.shape[3], dtype=bf)
        scr = m.scratch(l.spec.heads, l.spec.kv_heads, v.shape[3], t, m.attention_splits(l.spec, t, c.max_len, l.spec.chunk))
        P.flash_decode_scored(k, v, c.block_table, c.positions, l.mods, attn, scr, l.spec.heads, l.spec.dim, l.spec.vdim, raw=raw,
                              eps=eps, n_rows=t, chunk=l.spec.chunk, head_norm=True, bias=l.bias, inv_freq=l.inv_freq,
                              grow=l.grow, pdl=pdl)
        a = get("scan_a", t, r.w_o.k, dtype=bf)
        S.ssd_decode(raw[:, l.columns:], r.x_at, r.dt_at, r.conv_w, r.conv_b,
                     c.cache.layer_state(li, "conv") if r.spec.conv > 1 else None, r.dt_bias, r.a_log, r.skip, r.spec.groups,
                     c.slots, c.cache.layer_state(li, "ssd"), get("scan_o", t, r.w_o.k, dtype=torch.float32), r.norm, eps,
                     r.spec.norm_groups, a, pdl=pdl)
        return [(attn.view(t, -1), l.w_o, mw.left_scale), (a, r.w_o, mw.right_scale)]

    def _matvec_layers(self, c: StepContext) -> None:
        m, cfg, w, pdl, t = self.model, self.model.cfg, self.model.w, self.pdl, c.t
        eps, width, f32 = cfg.norm_eps, cfg.width, torch.float32
        get = c.bufs.get
        x = get("x", t, m.width_p, dtype=f32)
        P.embed_scaled(w.embed, self.tokens[:t], cfg.embedding_scale, x)
        for li, lw in enumerate(w.layers):
            mw, f = lw.mix, lw.mlp
            raw = get("raw32", t, mw.w_in.n, dtype=f32)
            ff = r = None
            if f is None:
                TN.twin_in(x, lw.norm1, eps, width, mw.w_in.w, raw, pdl=pdl)
            elif isinstance(f, DenseFfWeights):
                act = get("ff", t, f.w_down.k, dtype=torch.bfloat16)
                TN.twin_in(x, lw.norm1, eps, width, mw.w_in.w, raw, lw.norm2, f.w_gu.w, act, f.spec.limit, pdl=pdl)
                ff = (act, f.w_down, w.ones)
            else:
                r, h2 = m.routing(f, c), get("h2_32", t, m.width_p, dtype=f32)
                TN.twin_in_router(x, lw.norm1, eps, width, mw.w_in.w, raw, lw.norm2, f.router, f.correction,
                                  get("route_z", t, f.spec.experts, dtype=f32), h2, self.ticket, r, pdl=pdl)
            terms = self._mixer(li, mw, raw, c) + ([] if ff is None else [ff])
            for i in range(0, len(terms), 2):
                a, wa, sa = terms[i]
                b, wb, sb = terms[i + 1] if i + 1 < len(terms) else (None, None, None)
                P.gemv_out_add(a, wa.w, sa, b, None if wb is None else wb.w, sb, x, pdl=pdl)
            if r is not None:
                n = f.w_down.k
                act = get("moe_act", t, f.spec.top, n, dtype=torch.bfloat16).view(t * f.spec.top, n)
                R.postnorm_expert(h2, f.w_gu.w, f.spec.limit, r, act, pdl=pdl)
                # the weighted outputs beside one times the residual itself, which is where they go
                R.expert_out(act, f.w_down.w, R.Routing(r.idx, r.weights, w.ones, r.counts, r.offsets, r.row_of_pair), x, x, pdl=pdl)
        P.norm_in_proj(x, w.final_norm, eps, width, w.lm_head.w, cfg.vocab_size, 0.0, 0.0, self.logits[:t], None, pdl=pdl)
