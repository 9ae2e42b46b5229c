"""Nugosun: a decoder whose mixer and feed-forward read the same fp32 residual through norms of their own and are both
added to it. Mixers: latent attention with a query latent (layers may read an earlier layer's cached rows), gated
linear attention, and pairs of chunked attention and state-space heads whose weighted outputs are summed; the
feed-forward is dense or routed SwiGLU. The embedding table is the LM head, too.

The cache holds pages for the attention layers that own rows and, per sequence, one fp32 row of recurrent state
(``PagedKvCache``'s ``layer_states``): the matrix states and the inputs a convolution carries over. Widths that are
not multiples of eight are padded with zeros when the weights are built, so every kernel sees aligned rows.

Prompts and mixed batches run through ``forward_batch`` (a ragged batch), decode steps through ``TwinNormDecode`` (one
CUDA graph per step). Everything runs on this package's CUDA kernels, in bf16 or (``dtype=torch.float32``) in true
32-bit; there is no CPU path."""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Dict, List, Optional, Tuple, Union

import torch

from ..config import (ChosenFfSpec, ChunkedAttentionSpec, GlaSpec, LatentAttentionSpec, NugosunConfig, PairSpec, RotarySpec,
                      StateSpaceSpec, SwigluFfSpec, TwinNormLayerSpec)
from ..kv.paged import PagedKvCache
from ..ops import parallel_block as P
from ..ops import post_norm as N
from ..ops import routed as R
from ..ops import scan as S
from ..ops import twin_norm as TN
from ..ops.parallel_block import ScoreMods, pad8
from ..ops.post_norm import pad_to
from ..ops.weights import LinearWeight, W_BF16
from .ragged_model import (Buffers, DenseFfWeights, LatentWeights, RaggedModel, RoutedFfWeights, StepContext,
                           WeightBuilder, check_tensors, latent_row, save_checkpoint, weight_bytes)  # noqa: F401
from .weights import ParallelLayout

Term = Tuple[torch.Tensor, LinearWeight, torch.Tensor]       # activations, projection, per-column factor


def nugosun_tiny() -> NugosunConfig:
    """Test-size preset: every kind of sublayer, all sizes different."""
    rot = RotarySpec(5000.0, 20, {"factor": 3.0, "original": 40.0, "fast": 8.0, "slow": 0.5})
    lat = LatentAttentionSpec(5, 24, 16, 40, 72, 0.16, 5000.0, q_rank=52)
    return NugosunConfig(vocab_size=211, width=104, norm_eps=1e-5, embedding_scale=1.5, layers=[
        TwinNormLayerSpec(GlaSpec(3, 24, 40, 8.0, 6), ChosenFfSpec(7, 3, 40)),
        TwinNormLayerSpec(lat, SwigluFfSpec(136)),
        TwinNormLayerSpec(PairSpec(ChunkedAttentionSpec(6, 2, 32, 48, 0.2, rot, 15.0, 27),
                                   StateSpaceSpec(6, 16, 20, 2, 4, 3), 0.7, 1.3), ChosenFfSpec(5, 2, 72)),
        TwinNormLayerSpec(replace(lat, heads=3, dim=32, vdim=24, q_rank=36, kv_from=1), None),
        TwinNormLayerSpec(PairSpec(ChunkedAttentionSpec(2, 2, 24, 16, 0.25, RotarySpec(900.0, 24), 30.0, 9),
                                   StateSpaceSpec(2, 24, 33, 1, 2, 1), 1.1, 0.4), SwigluFfSpec(96))]).validate()


def nugosun_4096(num_layers: int = 32) -> NugosunConfig:
    """Layers of width 4096 (memory plan, benchmarks): in fours, latent attention + dense, gated linear attention +
    routed, a pair + routed, latent attention on the first one's rows + routed."""
    lat = LatentAttentionSpec(32, 128, 64, 128, 512, 192 ** -0.5, q_rank=1536)
    rot = RotarySpec(500000.0, 64, {"factor": 4.0, "original": 8192.0, "fast": 32.0, "slow": 1.0})
    pair = PairSpec(ChunkedAttentionSpec(32, 8, 128, 128, 128 ** -0.5, rot, 50.0, 1024),
                    StateSpaceSpec(64, 64, 128, 1, 4, 1), 1.0, 1.0)
    moe = ChosenFfSpec(32, 4, 3584)
    layers = [TwinNormLayerSpec(replace(lat, kv_from=i - 3) if i % 4 == 3 else (lat, GlaSpec(16, 128, 256, 16.0), pair)[i % 4],
                                SwigluFfSpec(14336) if i % 4 == 0 else moe) for i in range(num_layers)]
    return NugosunConfig(vocab_size=128256, width=4096, layers=layers, norm_eps=1e-6, name="nugosun-4096").validate()


# ------------------------------------------------------------------------------------------------
# Weights
# ------------------------------------------------------------------------------------------------
@dataclass
class GlaWeights:
    spec: GlaSpec
    w_in: LinearWeight               # [2 * qk_p + 2 * v_p + rank_p, width_p]: q | k | v | g | decay rank
    w_a2: torch.Tensor               # [pad8(heads * dim), rank_p]
    bias: torch.Tensor               # fp32 [heads * dim]
    norm: torch.Tensor               # fp32 [heads * vdim]
    w_o: LinearWeight                # [width_p, v_p]

    @property
    def qk_p(self) -> int:
        return pad8(self.spec.heads * self.spec.dim)

    @property
    def v_p(self) -> int:
        return self.w_o.k

    @property
    def at(self) -> Tuple[int, int, int, int, int]:
        """Columns of q, k, v, g and the decay rank in a row of w_in's result."""
        return 0, self.qk_p, 2 * self.qk_p, 2 * self.qk_p + self.v_p, 2 * (self.qk_p + self.v_p)


@dataclass
class StateSpaceWeights:
    spec: StateSpaceSpec
    conv_w: torch.Tensor             # fp32 [taps, channels], oldest first
    conv_b: torch.Tensor             # fp32 [channels]
    dt_bias: torch.Tensor            # fp32 [heads]
    a_log: torch.Tensor
    skip: torch.Tensor
    norm: torch.Tensor               # fp32 [inner]
    w_o: LinearWeight                # [width_p, pad8(inner)]

    @property
    def x_at(self) -> int:
        """Column of x | B | C (z is at 0)."""
        return pad8(self.spec.inner)

    @property
    def dt_at(self) -> int:
        return self.x_at + pad8(self.spec.channels)

    @property
    def columns(self) -> int:
        return self.dt_at + pad8(self.spec.heads)


@dataclass
class ChunkedWeights:
    spec: ChunkedAttentionSpec
    bias: torch.Tensor               # fp32 [q | k | v]
    inv_freq: torch.Tensor           # fp32 [rotated pairs]
    grow: float                      # factor of cos and sin
    mods: ScoreMods
    w_o: LinearWeight                # [width_p, heads * pad8(vdim)]

    @property
    def columns(self) -> int:
        m = self.spec
        return pad8((m.heads + m.kv_heads) * m.dim + m.kv_heads * m.vdim)


@dataclass
class PairWeights:
    spec: PairSpec
    w_in: LinearWeight               # [left columns + right columns, width_p]: q | k | v | z | x | B | C | dt
    left: ChunkedWeights
    right: StateSpaceWeights
    left_scale: torch.Tensor         # fp32 [width_p], all alike
    right_scale: torch.Tensor


@dataclass
class TwinNormLayerWeights:
    spec: TwinNormLayerSpec
    mix: Union[LatentWeights, GlaWeights, PairWeights]
    norm1: torch.Tensor              # fp32 [width_p], one already added
    mlp: Union[DenseFfWeights, RoutedFfWeights, None]
    norm2: Optional[torch.Tensor]


@dataclass
class NugosunWeights:
    cfg: NugosunConfig
    embed: torch.Tensor              # [vocab, width_p]; also the LM head's matrix
    layers: List[TwinNormLayerWeights]
    final_norm: torch.Tensor         # fp32 [width_p]
    lm_head: LinearWeight
    ones: torch.Tensor               # fp32 [width_p]
    layout: ParallelLayout
    vocab_base: int = 0

    def nbytes(self) -> int:
        pairs = [p for l in self.layers if isinstance(l.mix, PairWeights) for p in (l.mix.left, l.mix.right)]
        return weight_bytes(self, *[p for l in self.layers for p in (l, l.mix, l.mlp)], *pairs) - self.lm_head.nbytes()


def kv_shapes(cfg: NugosunConfig) -> List[Optional[tuple]]:
    """Per layer (kv heads, key row, value row) of the paged cache; latent rows are key and value at once, a layer that
    reads another's has none."""
    out: List[Optional[tuple]] = []
    for l in cfg.layers:
        m = l.mixer
        if isinstance(m, LatentAttentionSpec):
            out.append(latent_row(m))
        else:
            out.append((m.left.kv_heads, pad8(m.left.dim), pad8(m.left.vdim)) if isinstance(m, PairSpec) else None)
    return out


def state_shapes(cfg: NugosunConfig) -> List[Optional[Dict[str, tuple]]]:
    """Per layer what a sequence carries: the matrix states, and a convolution's last inputs (oldest first)."""
    out: List[Optional[Dict[str, tuple]]] = []
    for l in cfg.layers:
        m = l.mixer
        if isinstance(m, GlaSpec):
            out.append({"gla": (m.heads, m.dim, m.vdim)})
        elif isinstance(m, PairSpec):
            r = m.right
            out.append({"ssd": (r.heads, r.state, r.vdim), **({"conv": (r.conv - 1, r.channels)} if r.conv > 1 else {})})
        else:
            out.append(None)
    return out


def tensor_shapes(cfg: NugosunConfig) -> Dict[str, tuple]:
    """Checkpoint tensor names and shapes."""
    d = cfg.width
    out = {"embed": (cfg.vocab_size, d)}
    for i, l in enumerate(cfg.layers):
        m, p = l.mixer, f"l{i}.mix."
        out[f"l{i}.norm1"] = (d,)
        if isinstance(m, LatentAttentionSpec):
            out.update({p + "dq": (m.q_rank, d), p + "dq.norm": (m.q_rank,), p + "uq": (m.heads * (m.dim + m.rot_dim), m.q_rank),
                        p + "uk": (m.heads * m.dim, m.kv_rank), p + "uv": (m.heads * m.vdim, m.kv_rank),
                        p + "o": (d, m.heads * m.vdim)})
            if m.kv_from is None:
                out.update({p + "dkv": (m.kv_rank + m.rot_dim, d), p + "dkv.norm": (m.kv_rank,)})
        elif isinstance(m, GlaSpec):
            k, v = m.heads * m.dim, m.heads * m.vdim
            out.update({p + "q": (k, d), p + "k": (k, d), p + "v": (v, d), p + "g": (v, d), p + "a1": (m.decay_rank, d),
                        p + "a2": (k, m.decay_rank), p + "a2.b": (k,), p + "norm": (m.vdim,), p + "o": (d, v)})
        else:
            a, s, q, r = m.left, m.right, p + "left.", p + "right."
            for n, rows in (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim)):
                out.update({q + n: (rows, d), f"{q}{n}.b": (rows,)})
            out.update({q + "o": (d, a.heads * a.vdim), r + "in": (s.inner + s.channels + s.heads, d),
                        r + "conv": (s.channels, s.conv), r + "conv.b": (s.channels,), r + "dt_bias": (s.heads,),
                        r + "A_log": (s.heads,), r + "D": (s.heads,), r + "norm": (s.inner,), r + "o": (d, s.inner)})
        p = f"l{i}.mlp."
        if l.mlp is not None:
            out[f"l{i}.norm2"] = (d,)
            names = [p] if isinstance(l.mlp, SwigluFfSpec) else [f"{p}e{e}." for e in range(l.mlp.experts)]
            for q in names:
                out.update({q + "gate": (l.mlp.ff, d), q + "up": (l.mlp.ff, d), q + "down": (d, l.mlp.ff)})
            if isinstance(l.mlp, ChosenFfSpec):
                out.update({p + "router": (l.mlp.experts, d), p + "router.b": (l.mlp.experts,)})
    out["final.norm"] = (d,)
    return out


def random_tensors(cfg: NugosunConfig, seed: int = 0, device="cpu", dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Random checkpoint tensors of the design (projections scaled by 1 / sqrt(inputs))."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".", 1)[-1]
        x = torch.randn(*shape, generator=g, device=device, dtype=torch.float32 if len(shape) == 1 else dtype)
        if leaf in ("norm1", "norm2", "norm") and not name.endswith("mix.norm"):
            x = 0.2 * x                                  # weights around zero
        elif leaf.endswith("norm") or leaf.endswith(".D"):
            x = 1.0 + 0.2 * x
        elif leaf.endswith("A_log"):
            x = 0.5 + 0.5 * x
        elif leaf.endswith("dt_bias"):
            x = -3.0 + x
        elif leaf.endswith(".b"):
            x = 0.3 * x
        elif name != "embed" and len(shape) == 2:
            x = x * shape[1] ** -0.5
        out[name] = x.to(dtype)
    return out


def build_weights(cfg: NugosunConfig, tensors: Dict[str, torch.Tensor], device="cpu", dtype=torch.bfloat16
                  ) -> NugosunWeights:
    """Runtime weights from checkpoint tensors: projections merged and padded, per-channel vectors in
    fp32, everything on ``device``."""
    if dtype not in (torch.bfloat16, torch.float32):
        raise ValueError("Nugosun runs in bfloat16 or float32")
    ranks = {i: tensors[f"l{i}.mix.a1"].shape[0] for i, l in enumerate(cfg.layers)
             if isinstance(l.mixer, GlaSpec) and f"l{i}.mix.a1" in tensors}
    cfg = replace(cfg, layers=[replace(l, mixer=replace(l.mixer, decay_rank=ranks[i])) if i in ranks else l
                               for i, l in enumerate(cfg.layers)])
    check_tensors(tensors, tensor_shapes(cfg))
    b = WeightBuilder(tensors, cfg.width, device, dtype)
    wp = b.width_p

    def offset(name: str) -> torch.Tensor:
        """A norm's weight, stored around zero."""
        out = torch.zeros(wp, dtype=torch.float32, device=device)
        out[:cfg.width] = 1.0 + b.vec(tensors[name])
        return out

    def same(value: float) -> torch.Tensor:
        return torch.full((wp,), value, dtype=torch.float32, device=device)

    def gla(p: str, m: GlaSpec) -> GlaWeights:
        g = lambda n: tensors[p + n]                                     # noqa: E731
        k_p, v_p, rank_p = pad8(m.heads * m.dim), pad8(m.heads * m.vdim), pad_to(m.decay_rank, 16)
        w_in = torch.cat([b.mat([g(n)], rows, wp) for n, rows in (("q", k_p), ("k", k_p), ("v", v_p), ("g", v_p), ("a1", rank_p))])
        return GlaWeights(m, LinearWeight(W_BF16, w_in), b.mat([g("a2")], k_p, rank_p), b.vec(g("a2.b")),
                          b.vec(g("norm")).repeat(m.heads), b.lin([g("o")], wp, v_p))

    def pair(p: str, m: PairSpec) -> PairWeights:
        g = lambda n: tensors[p + n]                                     # noqa: E731
        a, s = m.left, m.right
        inv_freq, grow = TN.rotary_frequencies(a.rot.base, a.rot.dims, a.rot.scaling)
        left = ChunkedWeights(a, b.vec(torch.cat([g(f"left.{n}.b") for n in "qkv"])), b.vec(inv_freq), grow,
                              ScoreMods(a.scale, a.softcap), b.out_proj(g("left.o"), a.heads, a.vdim))
        right = StateSpaceWeights(s, b.vec(g("right.conv").t().contiguous()).view(s.conv, s.channels), b.vec(g("right.conv.b")),
                                  b.vec(g("right.dt_bias")), b.vec(g("right.A_log")), b.vec(g("right.D")), b.vec(g("right.norm")),
                                  b.lin([g("right.o")], wp, pad8(s.inner)))
        z, xbc, dt = torch.split(g("right.in"), [s.inner, s.channels, s.heads])
        w_in = torch.cat([b.mat([g(f"left.{n}") for n in "qkv"], left.columns, wp), b.mat([z], right.x_at, wp),
                          b.mat([xbc], right.dt_at - right.x_at, wp), b.mat([dt], pad8(s.heads), wp)])
        return PairWeights(m, LinearWeight(W_BF16, w_in), left, right, same(m.left_scale), same(m.right_scale))

    layers = []
    for i, spec in enumerate(cfg.layers):
        p, m, f = f"l{i}.", spec.mixer, spec.mlp
        mix = b.latent(p + "mix.", i, m) if isinstance(m, LatentAttentionSpec) else \
            gla(p + "mix.", m) if isinstance(m, GlaSpec) else pair(p + "mix.", m)
        mlp = None if f is None else b.dense(p + "mlp.", f) if isinstance(f, SwigluFfSpec) else \
            b.routed(p + "mlp.", f, "router.b")
        layers.append(TwinNormLayerWeights(spec, mix, offset(p + "norm1"), mlp, None if f is None else offset(p + "norm2")))
    table = b.lin([tensors["embed"]], cfg.vocab_size, wp)
    return NugosunWeights(cfg=cfg, embed=table.w, layers=layers, final_norm=offset("final.norm"), lm_head=table,
                          ones=same(1.0), layout=ParallelLayout())


# ------------------------------------------------------------------------------------------------
# Model
# ------------------------------------------------------------------------------------------------
class NugosunModel(RaggedModel):
    """One GPU's weights and the forward passes over them."""

    title = "Nugosun"

    def __init__(self, weights: NugosunWeights):
        heads = [m.left.heads if isinstance(m, PairSpec) else m.heads for m in (l.mixer for l in weights.cfg.layers)
                 if not isinstance(m, GlaSpec)]
        super().__init__(weights, kv_shapes(weights.cfg), state_shapes(weights.cfg), min(heads, default=1))

    @classmethod
    def from_config(cls, cfg: Optional[NugosunConfig] = None, seed: int = 0, device="cuda", dtype=torch.bfloat16
                    ) -> "NugosunModel":
        """Random-initialised model (default: the test-size preset)."""
        cfg = cfg or nugosun_tiny()
        gen_dev = device if torch.device(device).type == "cuda" and cfg.width >= 1024 else "cpu"
        return cls(build_weights(cfg, random_tensors(cfg, seed, gen_dev), device, dtype))

    def make_decode_engine(self, cache: PagedKvCache, max_batch: int, comm=None):
        from .twin_norm_decode import TwinNormDecode
        if comm is not None:
            raise ValueError("Nugosun runs on one GPU")
        return TwinNormDecode(self, cache, max_batch=max_batch)

    # ------------------------------------------------------------------ mixers: normed rows -> terms of the residual
    def latent_attention(self, li: int, mw: LatentWeights, h: torch.Tensor, c: StepContext) -> List[Term]:
        raw = N.linear(h, mw.w_in.w, c.bufs.get("raw", c.t, mw.w_in.n, dtype=self.dtype), pdl=c.pdl)
        return [(self.latent_core(li, mw, raw, c).view(c.t, -1), mw.w_o, self.w.ones)]

    def linear_attention(self, li: int, mw: GlaWeights, h: torch.Tensor, c: StepContext) -> List[Term]:
        m, t, dt, pdl = mw.spec, c.t, self.dtype, c.pdl
        raw = N.linear(h, mw.w_in.w, c.bufs.get("raw", t, mw.w_in.n, dtype=dt), pdl=pdl)
        q, k, v, g, low = (raw[:, a:] for a in mw.at)
        z = P.logits_f32(low[:, :mw.w_a2.shape[1]], mw.w_a2, c.bufs.get("decay", t, mw.qk_p, dtype=torch.float32))
        o = c.bufs.get("scan_o", t, mw.v_p, dtype=torch.float32)
        rec = c.bufs.get("scan_rec", t, m.heads, S.record(m.dim, m.vdim), dtype=torch.float32)
        S.gla_scan(q, k, v, z, mw.bias, m.tau, m.dim ** -0.5, c.cache.layer_state(li, "gla"), o, rec, runs=c.runs,
                   slots=None if c.runs is not None else c.slots, pdl=pdl)
        a = S.gated_norm(o, g, mw.norm, self.cfg.norm_eps, m.heads, c.bufs.get("scan_a", t, mw.v_p, dtype=dt), False, pdl=pdl)
        return [(a, mw.w_o, self.w.ones)]

    def chunked_attention(self, li: int, mw: ChunkedWeights, raw: torch.Tensor, c: StepContext) -> torch.Tensor:
        m, k, v = mw.spec, c.cache.k[li], c.cache.v[li]
        q = c.bufs.get("q", c.t, m.heads, k.shape[3], dtype=self.dtype)
        TN.rotary_norm_append(raw, mw.bias, mw.inv_freq, mw.grow, self.cfg.norm_eps, q, k, v, c.block_table, c.positions,
                              c.token_seq, m.heads, m.dim, m.vdim, pdl=c.pdl)
        return self.paged_attention(li, m, mw.mods, q, c, chunk=m.chunk)

    def state_space(self, li: int, mw: StateSpaceWeights, raw: torch.Tensor, c: StepContext) -> torch.Tensor:
        m, t, pdl = mw.spec, c.t, c.pdl
        o = c.bufs.get("scan_o", t, mw.w_o.k, dtype=torch.float32)
        rec = c.bufs.get("scan_rec", t, m.heads, S.record(m.state, m.vdim, True, m.heads // m.groups), dtype=torch.float32)
        S.ssd_scan(raw, mw.x_at, mw.dt_at, mw.conv_w, mw.conv_b, c.cache.layer_state(li, "conv") if m.conv > 1 else None,
                   mw.dt_bias, mw.a_log, mw.skip, m.groups, c.cache.layer_state(li, "ssd"), o, rec, c.slots, runs=c.runs, pdl=pdl)
        return S.gated_norm(o, raw, mw.norm, self.cfg.norm_eps, m.norm_groups,
                            c.bufs.get("scan_a", t, mw.w_o.k, dtype=self.dtype), True, pdl=pdl)

    def pair(self, li: int, mw: PairWeights, h: torch.Tensor, c: StepContext) -> List[Term]:
        raw = N.linear(h, mw.w_in.w, c.bufs.get("raw", c.t, mw.w_in.n, dtype=self.dtype), pdl=c.pdl)
        left = self.chunked_attention(li, mw.left, raw, c)
        right = self.state_space(li, mw.right, raw[:, mw.left.columns:], c)
        return [(left, mw.left.w_o, mw.left_scale), (right, mw.right.w_o, mw.right_scale)]

    # ------------------------------------------------------------------ layers
    def add_terms(self, x: torch.Tensor, terms: List[Term], c: StepContext) -> None:
        """x += every term's projection, two at a time."""
        for i in range(0, len(terms), 2):
            a, w, s = terms[i]
            b, w2, s2 = terms[i + 1] if i + 1 < len(terms) else (None, None, None)
            P.out_proj_add(a, w.w, s, b, None if w2 is None else w2.w, s2, x, pdl=c.pdl)

    def norms(self, li: int, x: torch.Tensor, h1: torch.Tensor, h2: torch.Tensor, experts=None, pdl: bool = False) -> None:
        """x += the experts' rows (if any); then the norms layer ``li`` reads (behind the last layer: none)."""
        lw = self.w.layers[li] if li < len(self.w.layers) else None
        if lw is None and experts is None:
            return
        n2 = None if lw is None else lw.norm2
        TN.twin_norm(x, None if lw is None else lw.norm1, None if lw is None else h1, n2, None if n2 is None else h2,
                     self.cfg.norm_eps, self.cfg.width, experts, pdl=pdl)

    def layer(self, li: int, acts, c: StepContext) -> None:
        """One layer over the fp32 residual ``x`` and its two norms, in place: the norms become the next layer's."""
        x, h1, h2 = acts
        lw = self.w.layers[li]
        mix = lw.mix
        if isinstance(mix, LatentWeights):
            terms = self.latent_attention(li, mix, h1, c)
        elif isinstance(mix, GlaWeights):
            terms = self.linear_attention(li, mix, h1, c)
        else:
            terms = self.pair(li, mix, h1, c)
        experts = None
        if isinstance(lw.mlp, DenseFfWeights):
            terms.append((self.dense_act(lw.mlp, h2, c), lw.mlp.w_down, self.w.ones))
        elif lw.mlp is not None:
            r = self.routing(lw.mlp, c)
            R.route_chosen(self.router_logits(lw.mlp, h2, c), lw.mlp.correction, r, pdl=c.pdl)
            experts = (self.expert_rows(lw.mlp, h2, r, c), r)
        self.add_terms(x, terms, c)
        self.norms(li + 1, x, h1, h2, experts, pdl=c.pdl)

    def start(self, tokens: torch.Tensor, bufs: Buffers, pdl: bool = False):
        """(fp32 residual, its norms for the first layer's mixer and feed-forward) of the tokens."""
        t = tokens.numel()
        x = bufs.get("x", t, self.width_p, dtype=torch.float32)
        h1, h2 = (bufs.get(n, t, self.width_p, dtype=self.dtype) for n in ("h", "h2"))
        P.embed_scaled(self.w.embed, tokens, self.cfg.embedding_scale, x, pdl=pdl)
        self.norms(0, x, h1, h2, pdl=pdl)
        return x, h1, h2
