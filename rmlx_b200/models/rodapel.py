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

import json
import os
from dataclasses import dataclass, replace
from typing import Dict, List, Optional, Sequence, Union

import torch

from .. import _lib
from ..config import (ClampedFfSpec, LatentAttentionSpec, PostNormLayerSpec, RodapelConfig, RoutedFfSpec,
                      WindowAttentionSpec, WkvSpec)
from ..kv.paged import PAGE, PagedKvCache
from ..ops import latent as L
from ..ops import parallel_block as P
from ..ops import post_norm as N
from ..ops import routed as R
from ..ops import wkv as W
from ..ops.decode import default_splits
from ..ops.gemm import GemmStatus
from ..ops.parallel_block import ScoreMods, pad8
from ..ops.post_norm import pad_to
from ..ops.weights import LinearWeight, W_BF16
from .ragged import Entry, RaggedBatch
from .weights import ParallelLayout

# Latent attention: batch entries of up to this many tokens attend to the cached latents; longer ones to keys
# and values expanded for their whole context (which costs about as much as 0.8 * kv_rank query tokens).
LATENT_ABSORB = 4
LATENT_ROW_PAD = 8       # unused values behind a latent cache row (csrc/kernels/mla_decode.cu)


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
class LatentWeights:
    spec: LatentAttentionSpec
    w_in: LinearWeight               # [rows, width_p]: q | latent | rotated key part
    c_norm: torch.Tensor             # fp32 [rank]
    w_uk: torch.Tensor               # [heads, lat_p, dim_p]: queries into the latent space
    w_uv: torch.Tensor               # [heads, vdim_p, lat_p]: attended latents to values
    w_ukv: LinearWeight              # [heads * (dim_p + vdim_p), lat_p]: latents to keys and values
    w_o: LinearWeight                # [width_p, heads * vdim_p]
    inv_freq: torch.Tensor           # fp32 [rotated pairs]
    mods: ScoreMods

    @property
    def dim_p(self) -> int:
        return pad8(self.spec.dim)

    @property
    def rot_p(self) -> int:
        return pad8(self.spec.rot_dim)

    @property
    def lat_p(self) -> int:
        return pad8(self.spec.kv_rank)

    @property
    def vdim_p(self) -> int:
        return pad8(self.spec.vdim)


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
class DenseFfWeights:
    spec: ClampedFfSpec
    w_gu: LinearWeight               # [2 * ff_p, width_p]: gate | up
    w_down: LinearWeight             # [width_p, ff_p]


@dataclass
class RoutedFfWeights:
    spec: RoutedFfSpec
    router: torch.Tensor             # [experts + identity, width_p]
    correction: torch.Tensor         # fp32 [experts + identity]
    w_gu: LinearWeight               # [experts, 2 * ff_p, width_p]
    w_down: LinearWeight             # [experts, rows, ff_p], rows: width rounded up to the tile width


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
        def size(v) -> int:
            if isinstance(v, LinearWeight):
                return v.nbytes()
            return v.numel() * v.element_size() if isinstance(v, torch.Tensor) else 0
        parts = [self] + [p for l in self.layers for p in (l, l.mix, l.mlp) if p is not None]
        return sum(size(v) for p in parts for v in vars(p).values())


def kv_shapes(cfg: RodapelConfig) -> List[Optional[tuple]]:
    """Per layer (kv heads, key row, value row) of the paged cache; latent rows are key and value at once."""
    out: List[Optional[tuple]] = []
    for l in cfg.layers:
        m = l.mixer
        if isinstance(m, WindowAttentionSpec):
            out.append((m.kv_heads, pad8(m.dim), pad8(m.vdim)))
        elif isinstance(m, LatentAttentionSpec):
            out.append((1, pad8(m.kv_rank) + pad8(m.rot_dim) + LATENT_ROW_PAD, 0))
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
    for name, shape in tensor_shapes(cfg).items():
        if name not in tensors:
            raise KeyError(f"checkpoint has no tensor {name!r}")
        if tuple(tensors[name].shape) != shape:
            raise ValueError(f"{name}: shape {tuple(tensors[name].shape)}, expected {shape}")
    width, wp = cfg.width, pad8(cfg.width)

    def dev(t: torch.Tensor) -> torch.Tensor:
        return t.to(device=device, dtype=dtype)

    def mat(parts, rows: int, cols: int) -> torch.Tensor:
        """Stack ``parts`` into a zero-padded [rows, cols] matrix."""
        out, at = torch.zeros(rows, cols, dtype=dtype, device=device), 0
        for t in parts:
            out[at:at + t.shape[0], :t.shape[1]] = dev(t)
            at += t.shape[0]
        return out

    def lin(parts, rows: int, cols: int) -> LinearWeight:
        return LinearWeight(W_BF16, mat(parts, rows, cols))

    def vec(t, n: Optional[int] = None) -> torch.Tensor:
        out = torch.zeros(n or t.numel(), dtype=torch.float32, device=device)
        out[:t.numel()] = t.reshape(-1).to(device=device, dtype=torch.float32)
        return out

    def out_proj(t, heads: int, vdim: int) -> LinearWeight:
        """Attention writes heads at stride pad8(vdim): the projection's columns are spread likewise."""
        wo = torch.zeros(wp, heads, pad8(vdim), dtype=dtype, device=device)
        wo[:width, :, :vdim] = dev(t).view(width, heads, vdim)
        return LinearWeight(W_BF16, wo.view(wp, -1))

    def mixer(i: int, m):
        g = lambda n: tensors[f"l{i}.mix.{n}"]                           # noqa: E731
        if isinstance(m, WindowAttentionSpec):
            rows = (m.heads + m.kv_heads) * m.dim + m.kv_heads * m.vdim + m.heads
            return WindowWeights(m, lin([g("q"), g("k"), g("v"), g("g")], pad8(rows), wp), vec(g("q.norm")),
                                 vec(g("k.norm")), out_proj(g("o"), m.heads, m.vdim), ScoreMods(m.scale))
        if isinstance(m, LatentAttentionSpec):
            rows = m.heads * (m.dim + m.rot_dim) + m.kv_rank + m.rot_dim
            uk = torch.zeros(m.heads, pad8(m.kv_rank), pad8(m.dim), dtype=dtype, device=device)
            uk[:, :m.kv_rank, :m.dim] = dev(g("uk")).view(m.heads, m.dim, m.kv_rank).transpose(1, 2)
            uv = torch.zeros(m.heads, pad8(m.vdim), pad8(m.kv_rank), dtype=dtype, device=device)
            uv[:, :m.vdim, :m.kv_rank] = dev(g("uv")).view(m.heads, m.vdim, m.kv_rank)
            ukv = torch.cat([uk.transpose(1, 2), uv], 1).reshape(-1, pad8(m.kv_rank)).contiguous()
            pairs = torch.arange(m.rot_dims // 2, dtype=torch.float64)
            return LatentWeights(m, lin([g("q"), g("dkv")], pad8(rows), wp), vec(g("dkv.norm")), uk, uv,
                                 LinearWeight(W_BF16, ukv), out_proj(g("o"), m.heads, m.vdim), vec(m.rot_base ** (-2.0 * pairs / max(m.rot_dims, 1))),
                                 ScoreMods(m.scale))
        n = m.heads * m.dim
        inner, rank_p = pad_to(n, 16), pad_to(m.decay_rank, 16)
        w_in = torch.cat([mat([g(s)], inner, wp) for s in "rkvg"] + [mat([g("w1")], rank_p, wp)])
        return WkvWeights(m, torch.stack([vec(g("mu." + s), wp) for s in W.SHIFT_PARTS]), LinearWeight(W_BF16, w_in),
                          mat([g("w2")], inner, rank_p), vec(g("w0")), vec(g("u")), vec(g("norm")), lin([g("o")], wp, inner))

    def feed_forward(i: int, f):
        p = f"l{i}.mlp."
        ffp = pad_to(f.ff, 64)

        def gate_up(q: str, out: torch.Tensor) -> None:
            out[:f.ff, :width], out[ffp:ffp + f.ff, :width] = dev(tensors[q + "gate"]), dev(tensors[q + "up"])

        if isinstance(f, ClampedFfSpec):
            gu = torch.zeros(2 * ffp, wp, dtype=dtype, device=device)
            gate_up(p, gu)
            return DenseFfWeights(f, LinearWeight(W_BF16, gu), lin([tensors[p + "down"]], wp, ffp))
        gu = torch.zeros(f.experts, 2 * ffp, wp, dtype=dtype, device=device)
        down = torch.zeros(f.experts, pad_to(wp, 128), ffp, dtype=dtype, device=device)
        for e in range(f.experts):
            gate_up(f"{p}e{e}.", gu[e])
            down[e, :width, :f.ff] = dev(tensors[f"{p}e{e}.down"])
        return RoutedFfWeights(f, mat([tensors[p + "router"]], f.experts + f.identity, wp), vec(tensors[p + "correction"]),
                               LinearWeight(W_BF16, gu), LinearWeight(W_BF16, down))

    layers = []
    for i, spec in enumerate(cfg.layers):
        layers.append(PostNormLayerWeights(
            spec, mixer(i, spec.mixer), vec(tensors[f"l{i}.norm1"], wp),
            None if spec.mlp is None else feed_forward(i, spec.mlp),
            None if spec.mlp is None else vec(tensors[f"l{i}.norm2"], wp)))
    return RodapelWeights(cfg=cfg, embed=dev(tensors["embed"]).contiguous(), embed_norm=vec(tensors["embed.norm"], wp),
                          layers=layers, final_norm=vec(tensors["final.norm"], wp),
                          lm_head=lin([tensors["head"]], cfg.vocab_size, wp), layout=ParallelLayout())


def save_checkpoint(model_dir: str, cfg: RodapelConfig, tensors: Dict[str, torch.Tensor]) -> None:
    """config.json and model.safetensors of a Rodapel model."""
    from safetensors.torch import save_file
    os.makedirs(model_dir, exist_ok=True)
    save_file({k: v.to(torch.bfloat16).contiguous().cpu() for k, v in tensors.items()},
              os.path.join(model_dir, "model.safetensors"))
    with open(os.path.join(model_dir, "config.json"), "w") as f:
        json.dump(cfg.to_json(), f, indent=1)


# ------------------------------------------------------------------------------------------------
# Model
# ------------------------------------------------------------------------------------------------
class Buffers:
    """Activations of up to ``rows`` tokens by name, shared by the layers. A name's storage grows to the
    widest layer that asks for it; storage that was handed out stays alive (a captured step may hold
    its address)."""

    def __init__(self, rows: int, device):
        self.rows, self.device = rows, device
        self._store: Dict[tuple, torch.Tensor] = {}
        self._old: List[torch.Tensor] = []

    def get(self, name: str, t: int, *shape: int, dtype) -> torch.Tensor:
        """[t, *shape], uninitialised except that fresh storage is zero."""
        per = 1
        for s in shape:
            per *= s
        buf = self._store.get((name, dtype))
        if buf is None or buf.numel() < self.rows * per:
            if buf is not None:
                self._old.append(buf)
            buf = self._store[name, dtype] = torch.zeros(self.rows * per, dtype=dtype, device=self.device)
        return buf[:t * per].view(t, *shape)

    def rows_of(self, name: str, n: int, *shape: int, dtype) -> torch.Tensor:
        """[n, *shape] where ``n`` is not bounded by the batch (expanded contexts): grows as needed."""
        per = 1
        for s in shape:
            per *= s
        buf = self._store.get((name, dtype))
        if buf is None or buf.numel() < n * per:
            self._store.pop((name, dtype), None)
            buf = self._store[name, dtype] = torch.zeros(n * per, dtype=dtype, device=self.device)
        return buf[:n * per].view(n, *shape)


@dataclass
class StepContext:
    """Where a batch's rows belong: everything the sublayers need beside the activations."""
    t: int
    bufs: Buffers
    cache: PagedKvCache
    block_table: torch.Tensor
    positions: torch.Tensor
    token_seq: Optional[torch.Tensor]        # row of block_table per token (None: its own row)
    slots: Optional[torch.Tensor]            # state slot per token
    runs: Optional[torch.Tensor]             # per sequence (first row, rows, slot, -); None: one row each
    batch: Optional[RaggedBatch] = None      # None: a decode step
    max_len: int = 0                         # decode step: longest context (plans KV splits)
    pdl: bool = False


class RodapelModel:
    """One GPU's weights and the forward passes over them."""

    # a step may hold prompt portions and decoded tokens together (``forward_batch``)
    mixed_batches = True

    def __init__(self, weights: RodapelWeights):
        self.w, self.cfg, self.layout = weights, weights.cfg, weights.layout
        self.device = weights.embed.device
        self.dtype = weights.embed.dtype
        self.width_p = pad8(self.cfg.width)
        self.allgather_logits = None
        self._bufs: Optional[Buffers] = None
        self._scratch: Dict[tuple, object] = {}
        latent = [l.mix for l in weights.layers if isinstance(l.mix, LatentWeights)]
        self._absorb = LATENT_ABSORB if self.device.type == "cuda" and any(map(self.latent_prefill, latent)) else None

    @classmethod
    def from_config(cls, cfg: Optional[RodapelConfig] = None, seed: int = 0, device="cuda", dtype=torch.bfloat16
                    ) -> "RodapelModel":
        """Random-initialised model (default: the test-size preset)."""
        cfg = cfg or rodapel_tiny()
        gen_dev = device if torch.device(device).type == "cuda" and cfg.width >= 1024 else "cpu"
        return cls(build_weights(cfg, random_tensors(cfg, seed, gen_dev), device, dtype))

    @classmethod
    def from_checkpoint(cls, model_dir: str, device="cuda", dtype=torch.bfloat16) -> "RodapelModel":
        from .registry import from_pretrained
        return from_pretrained(model_dir, device, dtype)

    # ------------------------------------------------------------------ cache
    def new_cache(self, num_blocks: int, max_seqs: int = 64, max_blocks_per_seq: Optional[int] = None,
                  dtype=None, kv_quant: Optional[str] = None) -> PagedKvCache:
        """``num_blocks`` pages of 16 tokens (page 0 is reserved). Without ``max_blocks_per_seq`` one
        sequence may take the whole pool, or ``cfg.max_seq_len`` tokens if that is set."""
        if kv_quant is not None:
            raise ValueError("Rodapel's attention kernels read 16- or 32-bit caches")
        if max_blocks_per_seq is None:
            max_blocks_per_seq = max(1, num_blocks - 1)
            if self.cfg.max_seq_len:
                max_blocks_per_seq = min(max_blocks_per_seq, (self.cfg.max_seq_len + PAGE - 1) // PAGE)
        shapes = kv_shapes(self.cfg)
        first = next((s for s in shapes if s is not None), (1, 8, 8))
        return PagedKvCache(num_blocks, len(shapes), first[0], first[1], dtype=dtype or self.dtype, device=self.device,
                            max_seqs=max_seqs, max_blocks_per_seq=max_blocks_per_seq, layer_shapes=shapes,
                            layer_states=state_shapes(self.cfg))

    def make_decode_engine(self, cache: PagedKvCache, max_batch: int, comm=None):
        from .post_norm_decode import PostNormDecode
        if comm is not None:
            raise ValueError("Rodapel runs on one GPU")
        return PostNormDecode(self, cache, max_batch=max_batch)

    # ------------------------------------------------------------------ sublayers: x -> output rows
    def scratch(self, heads: int, kv_heads: int, vdim_p: int, rows: int, splits: int) -> P.ScoredDecodeScratch:
        """Split-KV scratch, shared by every layer of the same head shape."""
        key = (heads, kv_heads, vdim_p, rows, splits)
        if key not in self._scratch:
            self._scratch[key] = P.ScoredDecodeScratch(rows, heads, kv_heads, vdim_p, splits, self.device)
        return self._scratch[key]

    def window_splits(self, m: WindowAttentionSpec, rows: int, max_len: int) -> int:
        if m.window:
            max_len = min(max_len, m.window + PAGE)
        return default_splits(rows, m.kv_heads, (m.heads // m.kv_heads + 15) // 16, max_len)

    def tensor_core_attention(self, m: WindowAttentionSpec) -> bool:
        return self.dtype == torch.bfloat16 and P.decode_scored_supported(pad8(m.dim), pad8(m.vdim)) and \
            P.prefill_scored_supported(pad8(m.dim), pad8(m.vdim))

    def window_attention(self, li: int, mw: WindowWeights, h: torch.Tensor, c: StepContext) -> torch.Tensor:
        m, t, dt, pdl = mw.spec, c.t, self.dtype, c.pdl
        k, v = c.cache.k[li], c.cache.v[li]
        raw = N.linear(h, mw.w_in.w, c.bufs.get("raw", t, mw.w_in.n, dtype=dt), pdl=pdl)
        q = c.bufs.get("q", t, m.heads, k.shape[3], dtype=dt)
        attn = c.bufs.get("attn", t, m.heads, v.shape[3], dtype=dt)
        N.head_norm_append(raw, mw.q_norm, mw.k_norm, self.cfg.norm_eps, q, k, v, c.block_table, c.positions, c.token_seq,
                           m.heads, m.dim, m.vdim, pdl=pdl)
        gate = raw[:, mw.gate_at:mw.gate_at + m.heads]
        b = c.batch
        if not self.tensor_core_attention(m):
            P.attention_any(q, k, v, c.block_table, c.positions, c.token_seq, mw.mods, attn, window=m.window, gate=gate,
                            pdl=pdl)
        elif b is None:
            s = self.scratch(m.heads, m.kv_heads, v.shape[3], t, self.window_splits(m, t, c.max_len))
            P.flash_decode_scored(k, v, c.block_table, c.positions, mw.mods, attn, s, m.heads, m.dim, m.vdim, q=q,
                                  n_rows=t, window=m.window, gate=gate, pdl=pdl)
        else:
            if b.tiles is not None:
                P.flash_prefill_scored(q, k, v, c.block_table, b.tiles, mw.mods, attn, window=m.window, lanes=b.lanes,
                                       gate=gate)
            if b.single is not None:
                n = len(b.single_host)
                s = self.scratch(m.heads, m.kv_heads, v.shape[3], n, self.window_splits(m, n, b.single_len))
                P.flash_decode_scored(k, v, c.block_table, c.positions, mw.mods, attn, s, m.heads, m.dim, m.vdim, q=q,
                                      rows=b.single, table_rows=c.token_seq, window=m.window, gate=gate)
        return self._output(attn.view(t, -1), mw.w_o, c)

    def latent_prefill(self, mw: LatentWeights) -> bool:
        return self.dtype == torch.bfloat16 and L.prefill_supported(mw.dim_p, mw.rot_p, mw.vdim_p)

    def absorbed_attention(self, mw: LatentWeights, pool: torch.Tensor, q: torch.Tensor, q_abs: torch.Tensor,
                           attn: torch.Tensor, c: StepContext, rows: Optional[torch.Tensor], longest: int) -> None:
        """Queries into the latent space, attention over the cached latents, attended latents to values."""
        m, pdl = mw.spec, c.pdl
        o_lat = c.bufs.get("o_lat", c.t, m.heads, mw.lat_p, dtype=self.dtype)
        N.head_gemv(mw.w_uk, q, q_abs, rows=rows, pdl=pdl)
        if self.dtype == torch.bfloat16 and (m.kv_rank, m.rot_dim) in L.DECODE_WIDTHS:
            n = c.t if rows is None else rows.numel()
            splits = L.decode_splits(n, m.heads, longest)
            key = ("latent", m.heads, mw.lat_p, n, splits)
            if key not in self._scratch:
                self._scratch[key] = L.LatentDecodeScratch(n, m.heads, splits, mw.lat_p, self.device)
            L.latent_decode(q_abs, pool, c.block_table, c.positions, m.scale, o_lat, self._scratch[key], rows=rows,
                            table_rows=c.token_seq, pdl=pdl)
        else:
            P.attention_any(q_abs, pool, pool, c.block_table, c.positions, c.token_seq, mw.mods, o_lat, rows=rows, pdl=pdl)
        N.head_gemv(mw.w_uv, o_lat, attn, rows=rows, pdl=pdl)

    def latent_core(self, li: int, mw: LatentWeights, raw: torch.Tensor, c: StepContext) -> torch.Tensor:
        """Everything between the two projections: raw [T, q | latent | key part] -> attention output rows."""
        m, t, dt, pdl = mw.spec, c.t, self.dtype, c.pdl
        pool, b = c.cache.k[li], c.batch
        q = c.bufs.get("q", t, m.heads, mw.dim_p + mw.rot_p, dtype=dt)
        q_abs = c.bufs.get("q_abs", t, m.heads, mw.lat_p + mw.rot_p, dtype=dt)
        attn = c.bufs.get("attn", t, m.heads, mw.vdim_p, dtype=dt)
        expand = b is not None and b.latent_tiles is not None and self.latent_prefill(mw)
        some_absorbed = not expand or b.absorbed is not None
        N.latent_append(raw, mw.c_norm, self.cfg.norm_eps, mw.inv_freq, q, q_abs if some_absorbed else None, pool,
                        c.block_table, c.positions, c.token_seq, m.heads, m.dim, m.rot_dim, m.kv_rank, mw.dim_p, mw.rot_p,
                        mw.lat_p, pdl=pdl)
        if expand:
            n = b.ctx_pages.shape[0] * PAGE
            ctx = c.bufs.rows_of("ctx", n, mw.lat_p, dtype=dt)
            kv = c.bufs.rows_of("ctx_kv", n, m.heads, mw.dim_p + mw.vdim_p, dtype=dt)
            L.latent_gather(pool, c.block_table, b.ctx_pages, ctx)
            N.linear(ctx, mw.w_ukv.w, kv.view(n, -1))
            L.flash_prefill_latent(q, kv, pool, mw.lat_p, c.block_table, b.latent_tiles, b.tile_ctx, m.scale, attn, mw.dim_p,
                                   lanes=b.latent_lanes)
        if some_absorbed:
            rows = b.absorbed if expand else None
            longest = c.max_len if b is None else b.absorbed_len if expand else max(p + l for p, l in zip(b.pos0, b.lens))
            self.absorbed_attention(mw, pool, q, q_abs, attn, c, rows, longest)
        return attn

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
        t, dt, ffp = c.t, self.dtype, fw.w_down.k
        scratch = c.bufs.get("gate_up", t, 2 * ffp, dtype=dt) if dt == torch.float32 else None
        act = N.gated_linear(h, fw.w_gu, fw.spec.limit, c.bufs.get("ff", t, ffp, dtype=dt), scratch, pdl=c.pdl)
        return self._output(act, fw.w_down, c)

    def routing(self, fw: RoutedFfWeights, c: StepContext) -> R.Routing:
        f, t = fw.spec, c.t
        i32 = dict(dtype=torch.int32)
        return R.Routing(c.bufs.get("route_idx", t, f.top, **i32), c.bufs.get("route_w", t, f.top, dtype=torch.float32),
                         c.bufs.get("route_id", t, dtype=torch.float32), c.bufs.get("route_counts", 1, f.experts, **i32)[0],
                         c.bufs.get("route_offsets", 1, f.experts + 1, **i32)[0],
                         c.bufs.get("route_rows", t, f.top, **i32))

    def routed_ff(self, lw: PostNormLayerWeights, fw: RoutedFfWeights, x: torch.Tensor, h: torch.Tensor,
                  c: StepContext) -> None:
        """Routed feed-forward with its norm and residual sum."""
        f, t, dt, pdl, ffp = fw.spec, c.t, self.dtype, c.pdl, fw.w_down.k
        logits = P.logits_f32(h, fw.router, c.bufs.get("route_z", t, fw.router.shape[0], dtype=torch.float32))
        r = self.routing(fw, c)
        R.route_corrected(logits, fw.correction, f.experts, r, pdl=pdl)
        xs = c.bufs.get("xs", t, f.top, self.width_p, dtype=dt).view(t * f.top, self.width_p)
        R.route_scatter(h, r, xs, pdl=pdl)
        act = c.bufs.get("moe_act", t, f.top, ffp, dtype=dt).view(t * f.top, ffp)
        y = c.bufs.get("moe_y", t, f.top, fw.w_down.n, dtype=dt).view(t * f.top, fw.w_down.n)
        scratch = c.bufs.get("moe_gu", t, f.top, 2 * ffp, dtype=dt).view(t * f.top, 2 * ffp) if dt == torch.float32 else None
        R.grouped_gated_ffn(xs, r.offsets, fw.w_gu, fw.w_down, f.limit, t, scratch, act, y, pdl=pdl)
        R.combine_post_norm(y, r, lw.norm2, self.cfg.norm_eps, self.cfg.width, x, h, pdl=pdl)

    def layer(self, li: int, x: torch.Tensor, h: torch.Tensor, c: StepContext) -> None:
        """One layer over the fp32 residual ``x`` and its copy ``h`` in the compute type, both in place."""
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

    def embed(self, tokens: torch.Tensor, bufs: Buffers, pdl: bool = False):
        """(fp32 residual, the same in the compute type) of the tokens."""
        t = tokens.numel()
        x = bufs.get("x", t, self.width_p, dtype=torch.float32)
        h = bufs.get("h", t, self.width_p, dtype=self.dtype)
        N.embed_norm(self.w.embed, tokens, self.w.embed_norm, self.cfg.norm_eps, x, h, pdl=pdl)
        return x, h

    def logits(self, x: torch.Tensor, h: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None,
               pdl: bool = False) -> torch.Tensor:
        """Final norm + LM head of fp32 residual rows [R, width_p] -> fp32 [R, vocab]."""
        w, r = self.w, x.shape[0]
        if out is None:
            out = torch.empty(r, self.cfg.vocab_size, dtype=torch.float32, device=self.device)
        if h is None:
            h = torch.empty(r, self.width_p, dtype=self.dtype, device=self.device)
        P.rms_norm_f32(x, w.final_norm, self.cfg.norm_eps, h, self.cfg.width, pdl=pdl)
        return P.logits_f32(h, w.lm_head.w, out=out)

    # ------------------------------------------------------------------ ragged batches
    def _buffers(self, rows: int) -> Buffers:
        if self._bufs is None or self._bufs.rows < rows:
            self._bufs = None
            self._bufs = Buffers(max(rows, 256), self.device)
        return self._bufs

    @torch.no_grad()
    def forward_batch(self, entries: Sequence[Entry], cache: PagedKvCache, observe=None) -> torch.Tensor:
        """Run the entries' tokens as one batch on top of what the cache holds; returns the wanted
        logits, fp32 [wanted, vocab], in the order of the entries and their ``want``. ``observe``:
        called with (layer, residual rows [T, width]) after every layer."""
        if self.device.type != "cuda":
            raise _lib.NativeError("Rodapel runs on this package's CUDA kernels only")
        batch = RaggedBatch.plan(entries, cache, min(l.mixer.heads for l in self.cfg.layers),
                                 self._absorb)
        for e, l in zip(batch.entries, batch.lens):
            cache.reserve(e.seq_id, l)
        batch.upload(self.device)
        bufs = self._buffers(batch.num_tokens)
        x, h = self.embed(batch.tokens, bufs)
        c = StepContext(batch.num_tokens, bufs, cache, cache.block_table, batch.positions, batch.token_seq, batch.token_seq,
                        batch.runs, batch)
        for li in range(len(self.w.layers)):
            self.layer(li, x, h, c)
            if observe is not None:
                observe(li, x[:, :self.cfg.width])
        for e, l in zip(batch.entries, batch.lens):
            cache.commit(e.seq_id, l)
        if not batch.want_host:
            return torch.empty(0, self.cfg.vocab_size, dtype=torch.float32, device=self.device)
        return self.logits(x.index_select(0, batch.want.long()))

    # ------------------------------------------------------------------ one-sequence conveniences
    @torch.no_grad()
    def prefill(self, token_ids: torch.Tensor, cache: PagedKvCache, seq_id: int, all_logits: bool = False,
                chunk: int = 8192) -> torch.Tensor:
        """Run a prompt (or a chunk of one); logits of the last token, [1, vocab], or of every position."""
        toks = token_ids.tolist()
        parts = []
        for lo in range(0, len(toks), chunk):
            part = toks[lo:lo + chunk]
            last = lo + chunk >= len(toks)
            want = range(len(part)) if all_logits else ([len(part) - 1] if last else ())
            parts.append(self.forward_batch([Entry(seq_id, part, want)], cache))
        GemmStatus.check(self.device)
        return torch.cat(parts, 0)

    def forward(self, token_ids: torch.Tensor, cache: Optional[PagedKvCache] = None,
                seq_ids: Optional[Sequence[int]] = None, last_only: bool = False) -> torch.Tensor:
        """``TransformerModel.forward``'s contract: equal counts of new tokens of every sequence."""
        toks = token_ids.tolist()
        if cache is None:
            cache, seq_ids = self.new_cache(len(toks) // PAGE + 2, max_seqs=1), [0]
            cache.add_sequence(0)
        n = len(toks) // len(seq_ids)
        want = [n - 1] if last_only else range(n)
        return self.forward_batch([Entry(s, toks[i * n:(i + 1) * n], want) for i, s in enumerate(seq_ids)], cache)

    @torch.no_grad()
    def generate_greedy(self, prompt: torch.Tensor, steps: int, cache: Optional[PagedKvCache] = None) -> List[int]:
        cache = cache or self.new_cache((prompt.numel() + steps) // PAGE + 2, max_seqs=1)
        cache.add_sequence(0)
        first = int(self.prefill(prompt, cache, 0)[0].argmax())
        if steps <= 1:
            return [first][:steps]
        eng = self.make_decode_engine(cache, 1)
        eng.bind([0], [first])
        return [first] + eng.generate(steps - 1)[0].tolist()

    def num_layers(self) -> int:
        return self.cfg.num_layers

    def config(self) -> RodapelConfig:
        return self.cfg
