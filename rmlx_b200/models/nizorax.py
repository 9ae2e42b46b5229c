"""Nizorax: a decoder whose sublayers sit between two layer norms, x <- x + norm_b(f(conv(norm(x)))), with a short causal
convolution over what each of them reads. Mixers: differential attention (two softmax maps per head over the same values,
sliding window) and lightning attention (linear attention with a constant decay per head); the feed-forward is dense with a
polynomial of normed powers, or routed SwiGLU with sigmoid scores, groups of experts and a shared expert. A range of layers
may run several times in a row with the same weights.

``NizoraxWeights.layers`` lists the layer *runs*: a looped layer's weights appear once per pass. The cache holds, per run,
pages for the attention layers (a key row is both maps' keys) and, per sequence, one fp32 row of recurrent state: the
matrix states and the inputs the convolutions carry over. Widths that are not multiples of eight are padded with zeros
when the weights are built, so every kernel sees aligned rows.

Prompts and mixed batches run through ``forward_batch`` (a ragged batch), decode steps through ``SandwichDecode`` (one CUDA
graph per step). Everything runs on this package's CUDA kernels, in bf16 or (``dtype=torch.float32``) in true 32-bit;
there is no CPU path."""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple, Union

import torch

from ..config import (DifferentialAttentionSpec, GroupedFfSpec, LightningSpec, LoopSpec, NizoraxConfig, PolyNormFfSpec,
                      RotarySpec, SandwichLayerSpec)
from ..kv.paged import PagedKvCache
from ..ops import parallel_block as P
from ..ops import post_norm as N
from ..ops import routed as R
from ..ops import sandwich as W
from ..ops import scan as S
from ..ops import twin_norm as TN
from ..ops.parallel_block import MapDiff, ScoreMods, pad8
from ..ops.post_norm import pad_to
from ..ops.weights import LinearWeight, W_BF16
from .ragged_model import (Buffers, RaggedModel, RoutedFfWeights, StepContext, WeightBuilder, check_tensors, save_checkpoint,
                           weight_bytes)  # noqa: F401
from .weights import ParallelLayout


def nizorax_tiny() -> NizoraxConfig:
    """Test-size preset: every kind of sublayer, all sizes different, a loop over two of the layers."""
    rot = RotarySpec(3000.0, 20, {"factor": 3.0, "original": 50.0, "high": 3.0, "low": 0.5})
    return NizoraxConfig(vocab_size=203, width=104, norm_eps=1e-5, embedding_scale=3.0, logit_scale=0.6, taps=3,
                         loop=LoopSpec(1, 3, 2), layers=[
        SandwichLayerSpec(LightningSpec(3, 24, 40, [0.5, 0.9, 0.99]), GroupedFfSpec(6, 2, 40, 3, 2, 1.5, 56)),
        SandwichLayerSpec(DifferentialAttentionSpec(6, 2, 28, 56, 0.2, rot, 0.35, 21), PolyNormFfSpec(136)),
        SandwichLayerSpec(LightningSpec(2, 36, 16, [0.7, 0.95]), None),
        SandwichLayerSpec(DifferentialAttentionSpec(3, 3, 40, 24, 0.15, RotarySpec(900.0, 40), 0.2, 50),
                          GroupedFfSpec(8, 3, 72, 4, 3, 0.8, 0))]).validate()


def nizorax_4096(num_layers: int = 32) -> NizoraxConfig:
    """Layers of width 4096 (memory plan, benchmarks): in fours, attention + dense, two lightning + routed, attention +
    routed; no loop."""
    rot = RotarySpec(500000.0, 64, {"factor": 8.0, "original": 8192.0, "high": 4.0, "low": 1.0})
    attn = DifferentialAttentionSpec(32, 8, 64, 128, 0.125, rot, 0.4, 1024)
    light = LightningSpec(32, 128, 128, [1.0 - 2.0 ** (-1 - i / 4) for i in range(32)])
    moe = GroupedFfSpec(32, 4, 3584, 8, 4, 1.0, 3584)
    layers = [SandwichLayerSpec(light if i % 4 in (1, 2) else attn, PolyNormFfSpec(14336) if i % 4 == 0 else moe)
              for i in range(num_layers)]
    return NizoraxConfig(vocab_size=128256, width=4096, layers=layers, norm_eps=1e-6, name="nizorax-4096").validate()


# ------------------------------------------------------------------------------------------------
# Weights
# ------------------------------------------------------------------------------------------------
@dataclass
class DiffAttentionWeights:
    spec: DifferentialAttentionSpec
    w_in: LinearWeight               # [rows, width_p]: q (head, map) | k (group, map) | v
    inv_freq: torch.Tensor           # fp32 [rotated pairs]
    mods: ScoreMods
    diff: MapDiff
    w_o: LinearWeight                # [width_p, heads * pad8(vdim)]


@dataclass
class LightningWeights:
    spec: LightningSpec
    w_in: LinearWeight               # [2 * qk_p + 2 * v_p, width_p]: q | k | v | g
    decay: torch.Tensor              # fp32 [heads]
    norm: torch.Tensor               # fp32 [heads * vdim]
    w_o: LinearWeight                # [width_p, v_p]

    @property
    def at(self) -> Tuple[int, int, int, int]:
        """Columns of q, k, v and g in a row of w_in's result."""
        qk_p, v_p = pad8(self.spec.heads * self.spec.dim), self.w_o.k
        return 0, qk_p, 2 * qk_p, 2 * qk_p + v_p


@dataclass
class PolyFfWeights:
    spec: PolyNormFfSpec
    w_up: LinearWeight               # [ff_p, width_p]
    act: torch.Tensor                # fp32 [4]
    w_down: LinearWeight             # [width_p, ff_p]


@dataclass
class SandwichLayerWeights:
    """Norms are fp32 [2, width_p] (weight, bias), convolutions fp32 [taps, width_p], oldest first; ``norm2``, ``post2`` and
    ``conv2`` are None without a feed-forward."""
    spec: SandwichLayerSpec
    mix: Union[DiffAttentionWeights, LightningWeights]
    norm1: torch.Tensor
    conv1: torch.Tensor
    post1: torch.Tensor
    mlp: Union[PolyFfWeights, RoutedFfWeights, None]
    norm2: Optional[torch.Tensor]
    conv2: Optional[torch.Tensor]
    post2: Optional[torch.Tensor]


@dataclass
class NizoraxWeights:
    cfg: NizoraxConfig
    embed: torch.Tensor              # [vocab, width_p]
    layers: List[SandwichLayerWeights]     # per run
    final_norm: torch.Tensor         # fp32 [2, width_p], times the logits' factor
    lm_head: LinearWeight            # [vocab, width_p]
    layout: ParallelLayout
    vocab_base: int = 0

    def nbytes(self) -> int:
        return weight_bytes(self, *[p for l in self.layers for p in (l, l.mix, l.mlp)])


def kv_shapes(cfg: NizoraxConfig) -> List[Optional[tuple]]:
    """Per run (kv heads, key row, value row) of the paged cache."""
    mixers = [cfg.layers[i].mixer for i in cfg.runs]
    return [(m.kv_heads, 2 * pad8(m.dim), pad8(m.vdim)) if isinstance(m, DifferentialAttentionSpec) else None for m in mixers]


def state_shapes(cfg: NizoraxConfig) -> List[Optional[Dict[str, tuple]]]:
    """Per run what a sequence carries: the matrix states, and the convolutions' last inputs (oldest first)."""
    out: List[Optional[Dict[str, tuple]]] = []
    for l in (cfg.layers[i] for i in cfg.runs):
        s: Dict[str, tuple] = {}
        if isinstance(l.mixer, LightningSpec):
            s["state"] = (l.mixer.heads, l.mixer.dim, l.mixer.vdim)
        if cfg.taps > 1:
            s["conv1"] = (cfg.taps - 1, pad8(cfg.width))
            if l.mlp is not None:
                s["conv2"] = (cfg.taps - 1, pad8(cfg.width))
        out.append(s or None)
    return out


def tensor_shapes(cfg: NizoraxConfig) -> Dict[str, tuple]:
    """Checkpoint tensor names and shapes."""
    d = cfg.width
    out: Dict[str, tuple] = {"embed": (cfg.vocab_size, d)}

    def norm(name: str) -> None:
        out.update({name: (d,), name + ".b": (d,)})

    for i, l in enumerate(cfg.layers):
        m, p = l.mixer, f"l{i}."
        norm(p + "norm1")
        norm(p + "norm1b")
        out[p + "canon1"] = (d, cfg.taps)
        if isinstance(m, DifferentialAttentionSpec):
            out.update({p + "mix.q": (m.heads * 2 * m.dim, d), p + "mix.k": (m.kv_heads * 2 * m.dim, d),
                        p + "mix.v": (m.kv_heads * m.vdim, d), p + "mix.o": (d, m.heads * m.vdim)})
            out.update({p + "mix." + n: (m.dim,) for n in ("lq1", "lk1", "lq2", "lk2")})
        else:
            k, v = m.heads * m.dim, m.heads * m.vdim
            out.update({p + "mix.q": (k, d), p + "mix.k": (k, d), p + "mix.v": (v, d), p + "mix.g": (v, d), p + "mix.o": (d, v),
                        p + "mix.norm": (v,)})
        f = l.mlp
        if f is None:
            continue
        norm(p + "norm2")
        norm(p + "norm2b")
        out[p + "canon2"] = (d, cfg.taps)
        if isinstance(f, PolyNormFfSpec):
            out.update({p + "mlp.up": (f.ff, d), p + "mlp.down": (d, f.ff), p + "mlp.act": (4,)})
            continue
        for q, ff in [(f"{p}mlp.e{e}.", f.ff) for e in range(f.experts)] + ([(p + "mlp.shared.", f.shared)] if f.shared else []):
            out.update({q + "gate": (ff, d), q + "up": (ff, d), q + "down": (d, ff)})
        out[p + "mlp.router"] = (f.experts, d)
    norm("final.norm")
    out["head"] = (cfg.vocab_size, d)
    return out


def random_tensors(cfg: NizoraxConfig, seed: int = 0, device="cpu", dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Random checkpoint tensors of the design (projections scaled by 1 / sqrt(inputs))."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        x = torch.randn(*shape, generator=g, device=device, dtype=torch.float32 if len(shape) == 1 else dtype)
        if leaf in ("norm", "norm1", "norm2", "norm1b", "norm2b"):
            x = 1.0 + 0.2 * x
        elif leaf == "b" or leaf in ("lq1", "lk1", "lq2", "lk2"):
            x = 0.2 * x
        elif leaf.startswith("canon"):
            x = 0.3 * x
        elif leaf != "embed" and len(shape) == 2:
            x = x * shape[1] ** -0.5
        out[name] = x.to(dtype)
    return out


def build_weights(cfg: NizoraxConfig, tensors: Dict[str, torch.Tensor], device="cpu", dtype=torch.bfloat16) -> NizoraxWeights:
    """Runtime weights from checkpoint tensors: projections merged and padded, per-channel vectors in
    fp32, everything on ``device``."""
    if dtype not in (torch.bfloat16, torch.float32):
        raise ValueError("Nizorax runs in bfloat16 or float32")
    check_tensors(tensors, tensor_shapes(cfg))
    b = WeightBuilder(tensors, cfg.width, device, dtype)
    wp = b.width_p

    def affine(name: str, factor: float = 1.0) -> torch.Tensor:
        return torch.stack([factor * b.vec(tensors[name + s], wp) for s in ("", ".b")])

    def conv(name: str) -> torch.Tensor:
        out = torch.zeros(cfg.taps, wp, dtype=torch.float32, device=device)
        out[:, :cfg.width] = tensors[name].to(device=device, dtype=torch.float32).t()
        return out

    def attention(p: str, m: DifferentialAttentionSpec) -> DiffAttentionWeights:
        g = lambda n: tensors[p + n]                                     # noqa: E731
        dot = lambda a, c: math.exp(float((g(a).double() * g(c).double()).sum()))      # noqa: E731
        rows = pad8((m.heads + m.kv_heads) * 2 * m.dim + m.kv_heads * m.vdim)
        return DiffAttentionWeights(m, b.lin([g(n) for n in "qkv"], rows, wp),
                                    b.vec(TN.rotary_frequencies(m.rot.base, m.rot.dims, m.rot.scaling)[0]), ScoreMods(m.scale),
                                    MapDiff(dot("lq1", "lk1") - dot("lq2", "lk2") + m.diff, 1.0 - m.diff, cfg.norm_eps),
                                    b.out_proj(g("o"), m.heads, m.vdim))

    def lightning(p: str, m: LightningSpec) -> LightningWeights:
        g = lambda n: tensors[p + n]                                     # noqa: E731
        k_p, v_p = pad8(m.heads * m.dim), pad8(m.heads * m.vdim)
        w_in = torch.cat([b.mat([g(n)], rows, wp) for n, rows in (("q", k_p), ("k", k_p), ("v", v_p), ("g", v_p))])
        return LightningWeights(m, LinearWeight(W_BF16, w_in), b.vec(torch.tensor(m.decay, dtype=torch.float64)), b.vec(g("norm")),
                                b.lin([g("o")], wp, v_p))

    def poly(p: str, f: PolyNormFfSpec) -> PolyFfWeights:
        ffp = pad_to(f.ff, 64)
        return PolyFfWeights(f, b.lin([tensors[p + "up"]], ffp, wp), b.vec(tensors[p + "act"]),
                             b.lin([tensors[p + "down"]], wp, ffp))

    def grouped(p: str, f: GroupedFfSpec) -> RoutedFfWeights:
        """Routed experts, then the shared one in equal slices (the activation is elementwise, so they add up to it)."""
        n, width = f.slices
        ffp = pad_to(width, 64)
        gu, down = b.zeros(f.experts + n, 2 * ffp, wp), b.zeros(f.experts + n, pad_to(wp, 128), ffp)

        def put(at: int, q: str, lo: int, hi: int) -> None:
            gu[at, :hi - lo, :cfg.width] = b.dev(tensors[q + "gate"][lo:hi])
            gu[at, ffp:ffp + hi - lo, :cfg.width] = b.dev(tensors[q + "up"][lo:hi])
            down[at, :cfg.width, :hi - lo] = b.dev(tensors[q + "down"][:, lo:hi])

        for e in range(f.experts):
            put(e, f"{p}e{e}.", 0, f.ff)
        for i in range(n):
            put(f.experts + i, p + "shared.", i * width, min((i + 1) * width, f.shared))
        return RoutedFfWeights(f, b.mat([tensors[p + "router"]], f.experts, wp), None, LinearWeight(W_BF16, gu),
                               LinearWeight(W_BF16, down), n)

    layers = []
    for i, spec in enumerate(cfg.layers):
        p, m, f = f"l{i}.", spec.mixer, spec.mlp
        mix = attention(p + "mix.", m) if isinstance(m, DifferentialAttentionSpec) else lightning(p + "mix.", m)
        mlp = None if f is None else poly(p + "mlp.", f) if isinstance(f, PolyNormFfSpec) else grouped(p + "mlp.", f)
        second = (None, None, None) if f is None else (affine(p + "norm2"), conv(p + "canon2"), affine(p + "norm2b"))
        layers.append(SandwichLayerWeights(spec, mix, affine(p + "norm1"), conv(p + "canon1"), affine(p + "norm1b"), mlp, *second))
    return NizoraxWeights(cfg=cfg, embed=b.mat([tensors["embed"]], cfg.vocab_size, wp), layers=[layers[i] for i in cfg.runs],
                          final_norm=affine("final.norm", cfg.logit_scale), lm_head=b.lin([tensors["head"]], cfg.vocab_size, wp),
                          layout=ParallelLayout())


# ------------------------------------------------------------------------------------------------
# Model
# ------------------------------------------------------------------------------------------------
class NizoraxModel(RaggedModel):
    """One GPU's weights and the forward passes over them."""

    title = "Nizorax"

    def __init__(self, weights: NizoraxWeights):
        # no head count for the prompt tiles: differential attention takes one tile of rows per block, in two maps
        super().__init__(weights, kv_shapes(weights.cfg), state_shapes(weights.cfg), 0)

    @classmethod
    def from_config(cls, cfg: Optional[NizoraxConfig] = None, seed: int = 0, device="cuda", dtype=torch.bfloat16) -> "NizoraxModel":
        """Random-initialised model (default: the test-size preset)."""
        cfg = cfg or nizorax_tiny()
        gen_dev = device if torch.device(device).type == "cuda" and cfg.width >= 1024 else "cpu"
        return cls(build_weights(cfg, random_tensors(cfg, seed, gen_dev), device, dtype))

    def make_decode_engine(self, cache: PagedKvCache, max_batch: int, comm=None):
        from .sandwich_decode import SandwichDecode
        if comm is not None:
            raise ValueError("Nizorax runs on one GPU")
        return SandwichDecode(self, cache, max_batch=max_batch)

    def carried(self, cache: PagedKvCache, li: int, name: str) -> Optional[torch.Tensor]:
        return cache.layer_state(li, name) if self.cfg.taps > 1 else None

    # ------------------------------------------------------------------ sublayers: input rows -> output rows
    def attention(self, li: int, mw: DiffAttentionWeights, h: torch.Tensor, c: StepContext) -> torch.Tensor:
        m, k, v = mw.spec, c.cache.k[li], c.cache.v[li]
        raw = N.linear(h, mw.w_in.w, c.bufs.get("raw", c.t, mw.w_in.n, dtype=self.dtype), pdl=c.pdl)
        q = c.bufs.get("q", c.t, m.heads, 2, pad8(m.dim), dtype=self.dtype)
        TN.rotary_norm_append(raw, None, mw.inv_freq, 1.0, 0.0, q, k, v, c.block_table, c.positions, c.token_seq, m.heads, m.dim,
                              m.vdim, neighbours=True, norm=False, maps=2, pdl=c.pdl)
        return self.paged_attention(li, m, mw.mods, q, c, window=m.window, diff=mw.diff)

    def lightning(self, li: int, mw: LightningWeights, h: torch.Tensor, c: StepContext) -> torch.Tensor:
        m, t, dt, pdl = mw.spec, c.t, self.dtype, c.pdl
        raw = N.linear(h, mw.w_in.w, c.bufs.get("raw", t, mw.w_in.n, dtype=dt), pdl=pdl)
        q, k, v, g = (raw[:, a:] for a in mw.at)
        o, state = c.bufs.get("scan_o", t, mw.w_o.k, dtype=torch.float32), c.cache.layer_state(li, "state")
        if c.runs is None:                                 # a token of every sequence
            W.lightning_step(raw, mw.at[1], mw.at[2], mw.decay, c.slots, state, o, pdl=pdl)
        else:
            rec = c.bufs.get("scan_rec", t, m.heads, S.record(m.dim, m.vdim, True), dtype=torch.float32)
            S.lightning_scan(q, k, v, mw.decay, state, o, rec, runs=c.runs, pdl=pdl)
        return S.gated_norm(o, g, mw.norm, self.cfg.norm_eps, 1, c.bufs.get("scan_a", t, mw.w_o.k, dtype=dt), False, sigmoid=True,
                            pdl=pdl)

    def poly(self, fw: PolyFfWeights, h: torch.Tensor, c: StepContext) -> torch.Tensor:
        z = N.linear(h, fw.w_up.w, c.bufs.get("ff", c.t, fw.w_up.n, dtype=self.dtype), pdl=c.pdl)
        return W.poly_norm(z, fw.act, self.cfg.norm_eps, fw.spec.ff, z, pdl=c.pdl)

    def groups(self, fw: RoutedFfWeights) -> R.RouteGroups:
        f = fw.spec
        return R.RouteGroups(f.groups, f.keep, f.scale, fw.always)

    # ------------------------------------------------------------------ layers
    def conv(self, li: int, name: str, w: torch.Tensor, h: torch.Tensor, hc: torch.Tensor, c: StepContext) -> None:
        W.short_conv(h, w, self.carried(c.cache, li, name), hc, c.slots, runs=c.runs, pdl=c.pdl)

    def layer(self, li: int, acts, c: StepContext) -> None:
        """One layer run over the fp32 residual ``x`` and its norm ``h``, in place: the norm becomes the next run's. In a decode
        step the convolution that follows a norm is part of its launch (the next run then finds its input convolved)."""
        x, h = acts
        lw, eps, width, pdl = self.w.layers[li], self.cfg.norm_eps, self.cfg.width, c.pdl
        after = self.w.layers[li + 1] if li + 1 < len(self.w.layers) else None
        step = c.batch is None and self.width_p <= W.step_max_width()
        hc = c.bufs.get("h_conv", c.t, self.width_p, dtype=self.dtype)
        out = lambda a, w: N.linear(a, w.w, c.bufs.get("y", c.t, self.width_p, dtype=self.dtype), pdl=pdl)    # noqa: E731

        def finish(y, post, norm, run, name, w, r=None) -> None:
            """x += post(y); the norm for what follows (of which ``step`` also does the convolution)."""
            if step and norm is not None:
                W.sandwich_step(x, y, post, norm, hc, eps, width, (w, self.carried(c.cache, run, name), c.slots), routing=r, pdl=pdl)
            else:
                W.sandwich_norm(x, y, post, norm, None if norm is None else h, eps, width, routing=r, pdl=pdl)

        follow = (None, li, "", None) if after is None else (after.norm1, li + 1, "conv1", after.conv1)
        if li == 0 or not step:
            self.conv(li, "conv1", lw.conv1, h, hc, c)
        mixer = self.attention if isinstance(lw.mix, DiffAttentionWeights) else self.lightning
        y = out(mixer(li, lw.mix, hc, c), lw.mix.w_o)
        if lw.mlp is None:
            finish(y, lw.post1, *follow)
            return
        finish(y, lw.post1, lw.norm2, li, "conv2", lw.conv2)
        if not step:
            self.conv(li, "conv2", lw.conv2, h, hc, c)
        if isinstance(lw.mlp, PolyFfWeights):
            finish(out(self.poly(lw.mlp, hc, c), lw.mlp.w_down), lw.post2, *follow)
        else:
            r = self.routing(lw.mlp, c)
            R.route_grouped(self.router_logits(lw.mlp, hc, c), self.groups(lw.mlp), r, pdl=pdl)
            finish(self.expert_rows(lw.mlp, hc, r, c), lw.post2, *follow, r)

    def start(self, tokens: torch.Tensor, bufs: Buffers, pdl: bool = False):
        """(fp32 residual, its norm for the first layer's mixer) of the tokens."""
        t = tokens.numel()
        x = bufs.get("x", t, self.width_p, dtype=torch.float32)
        h = bufs.get("h", t, self.width_p, dtype=self.dtype)
        P.embed_scaled(self.w.embed, tokens, self.cfg.embedding_scale, x, pdl=pdl)
        W.sandwich_norm(x, None, None, self.w.layers[0].norm1, h, self.cfg.norm_eps, self.cfg.width, pdl=pdl)
        return x, h

    def final_rows(self, x: torch.Tensor, h: torch.Tensor, pdl: bool = False) -> None:
        W.sandwich_norm(x, None, None, self.w.final_norm, h, self.cfg.norm_eps, self.cfg.width, pdl=pdl)
