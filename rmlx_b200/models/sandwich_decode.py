"""Cached decode of sandwich-norm decoders (``models/nizorax.py``): one row per sequence, one CUDA graph per step. In the
form of a few rows every sublayer starts with one launch that finishes the previous one (its output norm and the residual
sum), norms the residual and convolves it, and its projections read the result:

  attention           1. finish, norm, convolution   2. q | k | v projection   3. rotation, append, split-KV attention in two
                      maps, their difference and its norm   4. output projection
  lightning           1.   2. q | k | v | g projection   3. state   4. norm, gate, output projection
  dense feed-forward  1.   2. up projection   3. activation and down projection
  routed experts      1.   2. router and choice   3. gate / up of the chosen and the shared experts   4. weighted down"""
from __future__ import annotations

import torch

from ..ops import parallel_block as P
from ..ops import post_norm as N
from ..ops import routed as R
from ..ops import sandwich as W
from .layered_decode import LayeredDecode
from .nizorax import DiffAttentionWeights, PolyFfWeights
from .ragged_model import StepContext


class SandwichDecode(LayeredDecode):
    def _fits(self, lw) -> bool:
        m, f = lw.mix, lw.mlp
        if self.model.width_p > W.step_max_width() or N.max_rows(m.w_o.k) < 1:
            return False
        if isinstance(m, DiffAttentionWeights) and not self.model.tensor_core_attention(m.spec):
            return False
        if isinstance(f, PolyFfWeights):
            return N.max_rows(f.w_down.k) > 0
        return f is None or R.expert_decode_fits(f.w_down.k, f.spec.top + f.always)

    def _mixer(self, li: int, mw, h: torch.Tensor, y: torch.Tensor, c: StepContext) -> None:
        """y = the mixer's output rows."""
        m, t, pdl, eps, s = self.model, c.t, self.pdl, self.model.cfg.norm_eps, mw.spec
        get, f32 = c.bufs.get, torch.float32
        raw = N.rows_in(h, mw.w_in.w, get("raw32", t, mw.w_in.n, dtype=f32), pdl=pdl)
        if isinstance(mw, DiffAttentionWeights):
            k, v = c.cache.k[li], c.cache.v[li]
            attn = get("attn", t, s.heads, v.shape[3], dtype=torch.bfloat16)
            scr = m.scratch(2 * s.heads, s.kv_heads, v.shape[3], t, m.attention_splits(s, t, c.max_len, s.window))
            P.flash_decode_scored(k, v, c.block_table, c.positions, mw.mods, attn, scr, s.heads, s.dim, s.vdim, raw=raw, n_rows=t,
                                  window=s.window, head_norm=True, normed=False, inv_freq=mw.inv_freq, neighbours=True,
                                  diff=mw.diff, pdl=pdl)
            N.matvec_out(attn.view(t, -1), mw.w_o.w, y, pdl=pdl)
            return
        _, at_k, at_v, at_g = mw.at
        o = get("scan_o", t, mw.w_o.k, dtype=f32)
        W.lightning_step(raw, at_k, at_v, mw.decay, c.slots, c.cache.layer_state(li, "state"), o, pdl=pdl)
        W.gated_out(o, raw[:, at_g:], mw.norm, eps, mw.w_o.w, y, pdl=pdl)

    def _feed_forward(self, f, h: torch.Tensor, y: torch.Tensor, c: StepContext) -> None:
        m, t, pdl, get, f32 = self.model, c.t, self.pdl, c.bufs.get, torch.float32
        if isinstance(f, PolyFfWeights):
            z = N.rows_in(h, f.w_up.w, get("ff32", t, f.w_up.n, dtype=f32), pdl=pdl)
            W.poly_out(z, f.act, m.cfg.norm_eps, f.spec.ff, f.w_down.w, y, pdl=pdl)
            return
        r = m.routing(f, c)
        slots, n = r.idx.shape[1], f.w_down.k
        act = get("moe_act", t, slots, n, dtype=torch.bfloat16).view(t * slots, n)
        R.grouped_router(h, f.router, m.groups(f), get("route_z", t, f.spec.experts, dtype=f32), self.ticket, r, pdl=pdl)
        R.postnorm_expert(h, f.w_gu.w, f.spec.limit, r, act, pdl=pdl)
        R.expert_out(act, f.w_down.w, r, h, y, pdl=pdl)

    def _matvec_layers(self, c: StepContext) -> None:
        m, w, t, pdl = self.model, self.model.w, c.t, self.pdl
        eps, width, f32 = m.cfg.norm_eps, m.cfg.width, torch.float32
        x, h, y = (c.bufs.get(n, t, m.width_p, dtype=f32) for n in ("x", "h32", "y32"))
        P.embed_scaled(w.embed, self.tokens[:t], m.cfg.embedding_scale, x)
        pending = (None, None)                             # a sublayer's output and the norm it waits for
        for li, lw in enumerate(w.layers):
            W.sandwich_step(x, *pending, lw.norm1, h, eps, width, (lw.conv1, m.carried(c.cache, li, "conv1"), c.slots), pdl=pdl)
            self._mixer(li, lw.mix, h, y, c)
            pending = (y, lw.post1)
            if lw.mlp is not None:
                W.sandwich_step(x, *pending, lw.norm2, h, eps, width, (lw.conv2, m.carried(c.cache, li, "conv2"), c.slots), pdl=pdl)
                self._feed_forward(lw.mlp, h, y, c)
                pending = (y, lw.post2)
        W.sandwich_step(x, *pending, w.final_norm, h, eps, width, pdl=pdl)
        N.rows_in(h, w.lm_head.w, self.logits[:t], pdl=pdl)
