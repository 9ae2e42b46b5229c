"""Rodapel: a decoder whose layers mix three kinds of sublayers - grouped-query attention over a sliding
window (no positions, per-head norms, an output gate), latent attention (one cached latent and rotated
key part per token) and WKV recurrence (token shift, data-dependent decay) - with dense or routed
clamped-gate feed-forwards. Sublayers read the residual itself; the norms sit on their outputs.

The cache holds pages for the attention layers and, per sequence, one fp32 row of recurrent state for
the WKV layers (``PagedKvCache``'s ``layer_states``). Widths that are not multiples of eight are padded
with zeros when the weights are built, so every kernel sees aligned rows.

Prompts and mixed batches run through ``forward_batch`` (a ragged batch), decode steps through
``PostNormDecode`` (one CUDA graph per step). Everything runs on this package's CUDA kernels, in bf16 or
(``dtype=torch.float32``) in true 32-bit; there is no CPU path."""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Dict, List, Optional, Union

import torch

from ..config import (ClampedFfSpec, LatentAttentionSpec, PostNormLayerSpec, RodapelConfig, RoutedFfSpec,
                      WindowAttentionSpec, WkvSpec)
from ..kv.paged import PagedKvCache
from ..ops import parallel_block as P
from ..ops import post_norm as N
from ..ops import routed as R
from ..ops import wkv as W
from ..ops.parallel_block import ScoreMods, pad8
from ..ops.post_norm import pad_to
from ..ops.weights import LinearWeight, W_BF16
from .ragged_model import (LATENT_ABSORB, Buffers, DenseFfWeights, LatentWeights, RaggedModel, RoutedFfWeights,  # noqa: F401
                           StepContext, WeightBuilder, check_tensors, latent_row, save_checkpoint, weight_bytes)
from .weights import ParallelLayout


def rodapel_tiny() -> RodapelConfig:
    """Test-size preset: every kind of sublayer, all sizes different."""
    return RodapelConfig(vocab_size=211, width=104, norm_eps=1e-5, layers=[
        PostNormLayerSpec(WkvSpec(3, 32, 8), ClampedFfSpec(136, 2.0)),
        PostNormLayerSpec(WindowAttentionSpec(6, 2, 32, 40, 0.2, 24), RoutedFfSpec(6, 2, 3, 40, 1.5)),
        PostNormLayerSpec(LatentAttentionSpec(5, 24, 16, 32, 72, 0.16, 5000.0), ClampedFfSpec(96, 3.0)),
        PostNormLayerSpec(WindowAttentionSpec(2, 2, 24, 16, 0.25, 9), None)]).validate()


def rodapel_4096(num_layers: int = 32) -> RodapelConfig:
    """Layers of width 4096 (memory plan, benchmarks): in fours, windowed attention + dense, WKV + routed,
    latent attention + routed, windowed attention + routed."""
    win = WindowAttentionSpec(32, 8, 128, 128, 128 ** -0.5, 1024)
    lat = LatentAttentionSpec(32, 128, 64, 128, 512, 192 ** -0.5)
    moe = RoutedFfSpec(32, 8, 4, 3584, 7.0)
    four = [PostNormLayerSpec(win, ClampedFfSpec(14336, 7.0)), PostNormLayerSpec(WkvSpec(64, 64, 64), moe),
            PostNormLayerSpec(lat, moe), PostNormLayerSpec(win, moe)]
    return RodapelConfig(vocab_size=128256, width=4096, layers=(four * ((num_layers + 3) // 4))[:num_layers],
                         norm_eps=1e-6, name="rodapel-4096").validate()


# ------------------------------------------------------------------------------------------------
# Weights
# ------------------------------------------------------------------------------------------------
@dataclass
class WindowWeights:
    spec: WindowAttentionSpec
    w_in: LinearWeight               # [rows, width_p]: q | k | v | gate
    q_norm: torch.Tensor             # fp32 [dim]
    k_norm: torch.Tensor
    w_o: LinearWeight                # [width_p, heads * pad8(vdim)]
    mods: ScoreMods

    @property
    def gate_at(self) -> int:
        m = self.spec
        return (m.heads + m.kv_heads) * m.dim + m.kv_heads * m.vdim


@dataclass
class WkvWeights:
    spec: WkvSpec
    mu: torch.Tensor                 # fp32 [5, width_p] (r, k, v, g, w)
    w_in: LinearWeight               # [4 * inner_p + rank_p, width_p]: r | k | v | g | decay rank
    w2: torch.Tensor                 # [inner_p, rank_p]
    w0: torch.Tensor                 # fp32 [heads * dim]
    u: torch.Tensor                  # fp32 [heads * dim]
    norm: torch.Tensor               # fp32 [heads * dim]
    w_o: LinearWeight                # [width_p, inner_p]

    @property
    def inner_p(self) -> int:
        return self.w_o.k

    @property
    def rank_p(self) -> int:
        return self.w2.shape[1]

    def part(self, s: int) -> torch.Tensor:
        """Projection of shift part ``s`` (r, k, v, g; 4: the decay's first factor)."""
        at = s * self.inner_p
        return self.w_in.w[at:at + (self.inner_p if s < 4 else self.rank_p)]


@dataclass
class PostNormLayerWeights:
    spec: PostNormLayerSpec
    mix: Union[WindowWeights, LatentWeights, WkvWeights]
    norm1: torch.Tensor              # fp32 [width_p]
    mlp: Union[DenseFfWeights, RoutedFfWeights, None]
    norm2: Optional[torch.Tensor]


@dataclass
class RodapelWeights:
    cfg: RodapelConfig
    embed: torch.Tensor              # [vocab, width]
    embed_norm: torch.Tensor         # fp32 [width_p]
    layers: List[PostNormLayerWeights]
    final_norm: torch.Tensor         # fp32 [width_p]
    lm_head: LinearWeight            # [vocab, width_p]
    layout: ParallelLayout
    vocab_base: int = 0

    def nbytes(self) -> int:
        return weight_bytes(self, *[p for l in self.layers for p in (l, l.mix, l.mlp)])


def kv_shapes(cfg: RodapelConfig) -> List[Optional[tuple]]:
    """Per layer (kv heads, key row, value row) of the paged cache; latent rows are key and value at once."""
    out: List[Optional[tuple]] = []
    for l in cfg.layers:
        m = l.mixer
        if isinstance(m, WindowAttentionSpec):
            out.append((m.kv_heads, pad8(m.dim), pad8(m.vdim)))
        elif isinstance(m, LatentAttentionSpec):
            out.append(latent_row(m))
        else:
            out.append(None)
    return out


def state_shapes(cfg: RodapelConfig) -> List[Optional[Dict[str, tuple]]]:
    """Per layer what a sequence carries: the WKV state and the last token's residual row."""
    return [{"wkv": (l.mixer.heads, l.mixer.dim, l.mixer.dim), "prev": (pad8(cfg.width),)}
            if isinstance(l.mixer, WkvSpec) else None for l in cfg.layers]


def tensor_shapes(cfg: RodapelConfig) -> Dict[str, tuple]:
    """Checkpoint tensor names and shapes."""
    d = cfg.width
    out = {"embed": (cfg.vocab_size, d), "embed.norm": (d,)}
    for i, l in enumerate(cfg.layers):
        m, p = l.mixer, f"l{i}."
        out[p + "norm1"] = (d,)
        p += "mix."
        if isinstance(m, WindowAttentionSpec):
            out.update({p + "q": (m.heads * m.dim, d), p + "k": (m.kv_heads * m.dim, d), p + "v": (m.kv_heads * m.vdim, d),
                        p + "q.norm": (m.dim,), p + "k.norm": (m.dim,), p + "g": (m.heads, d),
                        p + "o": (d, m.heads * m.vdim)})
        elif isinstance(m, LatentAttentionSpec):
            out.update({p + "q": (m.heads * (m.dim + m.rot_dim), d), p + "dkv": (m.kv_rank + m.rot_dim, d),
                        p + "dkv.norm": (m.kv_rank,), p + "uk": (m.heads * m.dim, m.kv_rank),
                        p + "uv": (m.heads * m.vdim, m.kv_rank), p + "o": (d, m.heads * m.vdim)})
        else:
            n, rank = m.heads * m.dim, m.decay_rank
            out.update({p + "mu." + s: (d,) for s in W.SHIFT_PARTS})
            out.update({p + s: (n, d) for s in "rkvg"})
            out.update({p + "w1": (rank, d), p + "w2": (n, rank), p + "w0": (n,), p + "u": (m.heads, m.dim),
                        p + "norm": (n,), p + "o": (d, n)})
        p = f"l{i}.mlp."
        if l.mlp is not None:
            out[f"l{i}.norm2"] = (d,)
            names = [p] if isinstance(l.mlp, ClampedFfSpec) else [f"{p}e{e}." for e in range(l.mlp.experts)]
            for q in names:
                out.update({q + "gate": (l.mlp.ff, d), q + "up": (l.mlp.ff, d), q + "down": (d, l.mlp.ff)})
            if isinstance(l.mlp, RoutedFfSpec):
                n = l.mlp.experts + l.mlp.identity
                out.update({p + "router": (n, d), p + "correction": (n,)})
    out.update({"final.norm": (d,), "head": (cfg.vocab_size, d)})
    return out


def random_tensors(cfg: RodapelConfig, seed: int = 0, device="cpu", dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Random checkpoint tensors of the design (projections scaled by 1 / sqrt(inputs))."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.rsplit(".", 1)[-1]
        x = torch.randn(*shape, generator=g, device=device, dtype=torch.float32 if len(shape) == 1 else dtype)
        if leaf in ("norm", "norm1", "norm2"):
            x = 1.0 + 0.2 * x
        elif ".mu." in name:
            x = torch.sigmoid(x)
        elif leaf == "w0":
            x = -2.0 + 1.5 * x
        elif leaf == "u":
            x = 0.5 * x
        elif leaf == "correction":
            x = 0.1 * x
        elif len(shape) == 2 and name != "embed":
            x = x * shape[1] ** -0.5
        out[name] = x.to(dtype)
    return out


def build_weights(cfg: RodapelConfig, tensors: Dict[str, torch.Tensor], device="cpu", dtype=torch.bfloat16
                  ) -> RodapelWeights:
    """Runtime weights from checkpoint tensors: projections merged and padded, per-channel vectors in
    fp32, everything on ``device``."""
    if dtype not in (torch.bfloat16, torch.float32):
        raise ValueError("Rodapel runs in bfloat16 or float32")
    ranks = {i: tensors[f"l{i}.mix.w1"].shape[0] for i, l in enumerate(cfg.layers)
             if isinstance(l.mixer, WkvSpec) and f"l{i}.mix.w1" in tensors}
    cfg = replace(cfg, layers=[replace(l, mixer=replace(l.mixer, decay_rank=ranks[i])) if i in ranks else l
                               for i, l in enumerate(cfg.layers)])
    check_tensors(tensors, tensor_shapes(cfg))
    b = WeightBuilder(tensors, cfg.width, device, dtype)
    wp, vec, lin, mat = b.width_p, b.vec, b.lin, b.mat

    def mixer(i: int, m):
        g = lambda n: tensors[f"l{i}.mix.{n}"]                           # noqa: E731
        if isinstance(m, WindowAttentionSpec):
            rows = (m.heads + m.kv_heads) * m.dim + m.kv_heads * m.vdim + m.heads
            return WindowWeights(m, lin([g("q"), g("k"), g("v"), g("g")], pad8(rows), wp), vec(g("q.norm")),
                                 vec(g("k.norm")), b.out_proj(g("o"), m.heads, m.vdim), ScoreMods(m.scale))
        if isinstance(m, LatentAttentionSpec):
            return b.latent(f"l{i}.mix.", i, m)
        n = m.heads * m.dim
        inner, rank_p = pad_to(n, 16), pad_to(m.decay_rank, 16)
        w_in = torch.cat([mat([g(s)], inner, wp) for s in "rkvg"] + [mat([g("w1")], rank_p, wp)])
        return WkvWeights(m, torch.stack([vec(g("mu." + s), wp) for s in W.SHIFT_PARTS]), LinearWeight(W_BF16, w_in),
                          mat([g("w2")], inner, rank_p), vec(g("w0")), vec(g("u")), vec(g("norm")), lin([g("o")], wp, inner))

    def feed_forward(i: int, f):
        p = f"l{i}.mlp."
        return b.dense(p, f) if isinstance(f, ClampedFfSpec) else b.routed(p, f, "correction")

    layers = []
    for i, spec in enumerate(cfg.layers):
        layers.append(PostNormLayerWeights(
            spec, mixer(i, spec.mixer), vec(tensors[f"l{i}.norm1"], wp),
            None if spec.mlp is None else feed_forward(i, spec.mlp),
            None if spec.mlp is None else vec(tensors[f"l{i}.norm2"], wp)))
    return RodapelWeights(cfg=cfg, embed=b.dev(tensors["embed"]).contiguous(), embed_norm=vec(tensors["embed.norm"], wp),
                          layers=layers, final_norm=vec(tensors["final.norm"], wp),
                          lm_head=lin([tensors["head"]], cfg.vocab_size, wp), layout=ParallelLayout())


# ------------------------------------------------------------------------------------------------
# Model
# ------------------------------------------------------------------------------------------------
class RodapelModel(RaggedModel):
    """One GPU's weights and the forward passes over them."""

    title = "Rodapel"

    def __init__(self, weights: RodapelWeights):
        super().__init__(weights, kv_shapes(weights.cfg), state_shapes(weights.cfg),
                         min(l.mixer.heads for l in weights.cfg.layers))

    @classmethod
    def from_config(cls, cfg: Optional[RodapelConfig] = None, seed: int = 0, device="cuda", dtype=torch.bfloat16
                    ) -> "RodapelModel":
        """Random-initialised model (default: the test-size preset)."""
        cfg = cfg or rodapel_tiny()
        gen_dev = device if torch.device(device).type == "cuda" and cfg.width >= 1024 else "cpu"
        return cls(build_weights(cfg, random_tensors(cfg, seed, gen_dev), device, dtype))

    def make_decode_engine(self, cache: PagedKvCache, max_batch: int, comm=None):
        from .post_norm_decode import PostNormDecode
        if comm is not None:
            raise ValueError("Rodapel runs on one GPU")
        return PostNormDecode(self, cache, max_batch=max_batch)

    # ------------------------------------------------------------------ sublayers: x -> output rows
    def window_attention(self, li: int, mw: WindowWeights, h: torch.Tensor, c: StepContext) -> torch.Tensor:
        m, t, dt, pdl = mw.spec, c.t, self.dtype, c.pdl
        k, v = c.cache.k[li], c.cache.v[li]
        raw = N.linear(h, mw.w_in.w, c.bufs.get("raw", t, mw.w_in.n, dtype=dt), pdl=pdl)
        q = c.bufs.get("q", t, m.heads, k.shape[3], dtype=dt)
        N.head_norm_append(raw, mw.q_norm, mw.k_norm, self.cfg.norm_eps, q, k, v, c.block_table, c.positions, c.token_seq,
                           m.heads, m.dim, m.vdim, pdl=pdl)
        attn = self.paged_attention(li, m, mw.mods, q, c, window=m.window, gate=raw[:, mw.gate_at:mw.gate_at + m.heads])
        return self._output(attn, mw.w_o, c)

    def latent_attention(self, li: int, mw: LatentWeights, h: torch.Tensor, c: StepContext) -> torch.Tensor:
        raw = N.linear(h, mw.w_in.w, c.bufs.get("raw", c.t, mw.w_in.n, dtype=self.dtype), pdl=c.pdl)
        return self._output(self.latent_core(li, mw, raw, c).view(c.t, -1), mw.w_o, c)

    def time_mix(self, li: int, mw: WkvWeights, x: torch.Tensor, c: StepContext) -> torch.Tensor:
        m, t, dt, pdl, inner = mw.spec, c.t, self.dtype, c.pdl, mw.inner_p
        state, prev = c.cache.layer_state(li, "wkv"), c.cache.layer_state(li, "prev")
        parts = len(W.SHIFT_PARTS)
        mix = c.bufs.get("mix", t, parts, self.width_p, dtype=dt).view(parts, t, self.width_p)
        W.token_shift(x, mw.mu, prev, c.slots, c.runs is None, mix, pdl=pdl)
        rkvg = c.bufs.get("rkvg", t, 4, inner, dtype=dt).view(4, t, inner)
        for s in range(4):
            N.linear(mix[s], mw.part(s), rkvg[s], pdl=pdl)
        low = P.logits_f32(mix[4], mw.part(4), c.bufs.get("low", t, mw.rank_p, dtype=torch.float32))
        low_t = N.tanh_rows(low, c.bufs.get("low_t", t, mw.rank_p, dtype=dt), pdl=pdl)
        decay = P.logits_f32(low_t, mw.w2, c.bufs.get("decay", t, inner, dtype=torch.float32))
        o = c.bufs.get("wkv_o", t, inner, dtype=torch.float32)
        rec = c.bufs.get("wkv_rec", t, m.heads, W.record(m.dim), dtype=torch.float32)
        W.wkv_scan(rkvg[0], rkvg[1], rkvg[2], decay, mw.w0, mw.u, state, prev, x, o, rec, runs=c.runs,
                   slots=None if c.runs is not None else c.slots, pdl=pdl)
        a = c.bufs.get("wkv_a", t, inner, dtype=dt)
        W.wkv_finish(o, rkvg[3], mw.norm, self.cfg.norm_eps, m.heads, m.dim, a, pdl=pdl)
        return self._output(a, mw.w_o, c)

    def _output(self, a: torch.Tensor, w: LinearWeight, c: StepContext) -> torch.Tensor:
        """A sublayer's last projection, fp32 rows (the norm that follows reads them unrounded)."""
        return P.logits_f32(a, w.w, c.bufs.get("y", c.t, w.n, dtype=torch.float32))

    def dense_ff(self, fw: DenseFfWeights, h: torch.Tensor, c: StepContext) -> torch.Tensor:
        return self._output(self.dense_act(fw, h, c), fw.w_down, c)

    def routed_ff(self, lw: PostNormLayerWeights, fw: RoutedFfWeights, x: torch.Tensor, h: torch.Tensor,
                  c: StepContext) -> None:
        """Routed feed-forward with its norm and residual sum."""
        r = self.routing(fw, c)
        R.route_corrected(self.router_logits(fw, h, c), fw.correction, fw.spec.experts, r, pdl=c.pdl)
        y = self.expert_rows(fw, h, r, c)
        R.combine_post_norm(y, r, lw.norm2, self.cfg.norm_eps, self.cfg.width, x, h, pdl=c.pdl)

    def layer(self, li: int, acts, c: StepContext) -> None:
        """One layer over the fp32 residual ``x`` and its copy ``h`` in the compute type, both in place."""
        x, h = acts
        lw, eps, width = self.w.layers[li], self.cfg.norm_eps, self.cfg.width
        if isinstance(lw.mix, WindowWeights):
            y = self.window_attention(li, lw.mix, h, c)
        elif isinstance(lw.mix, LatentWeights):
            y = self.latent_attention(li, lw.mix, h, c)
        else:
            y = self.time_mix(li, lw.mix, x, c)
        N.post_norm_add(y, lw.norm1, eps, width, x, h, pdl=c.pdl)
        if isinstance(lw.mlp, DenseFfWeights):
            N.post_norm_add(self.dense_ff(lw.mlp, h, c), lw.norm2, eps, width, x, h, pdl=c.pdl)
        elif lw.mlp is not None:
            self.routed_ff(lw, lw.mlp, x, h, c)

    def start(self, tokens: torch.Tensor, bufs: Buffers, pdl: bool = False):
        """(fp32 residual, the same in the compute type) of the tokens."""
        t = tokens.numel()
        x = bufs.get("x", t, self.width_p, dtype=torch.float32)
        h = bufs.get("h", t, self.width_p, dtype=self.dtype)
        N.embed_norm(self.w.embed, tokens, self.w.embed_norm, self.cfg.norm_eps, x, h, pdl=pdl)
        return x, h
