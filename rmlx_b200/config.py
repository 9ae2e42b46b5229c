"""Typed configuration structs with ``validate()``.

Field names and defaults follow the reference's config structs so a user can carry settings over:
``TransformerConfig`` / ``FeedForwardType`` (crates/rmlx-nn/src/transformer.rs:38-109),
``MoeConfig`` (crates/rmlx-nn/src/moe.rs:114-132), ``AttentionConfig``
(crates/rmlx-nn/src/attention.rs:1790-1796), ``MlaConfig`` (crates/rmlx-nn/src/mla.rs:47-66),
``SchedulerConfig`` (crates/rmlx-nn/src/scheduler.rs:19-31), ``SamplerConfig``
(crates/rmlx-nn/src/sampler.rs:21-64), ``InitConfig`` (crates/rmlx-distributed/src/init.rs:38-95).
"""
from __future__ import annotations

import dataclasses
from dataclasses import dataclass, field
from typing import Optional


class ConfigError(ValueError):
    pass


def _require(cond: bool, msg: str) -> None:
    if not cond:
        raise ConfigError(msg)


@dataclass
class MoeConfig:
    num_experts: int
    num_experts_per_token: int
    hidden_dim: int
    intermediate_dim: int
    capacity_factor: float = 1.0      # only used by the capacity-limited (reference-style) dispatch
    enable_fp8: bool = False          # FP8 (E4M3, per-token scale) dispatch payload
    num_shared_experts: int = 0       # DeepSeek-style always-on experts
    shared_intermediate_dim: int = 0
    norm_topk_prob: bool = True

    def validate(self) -> "MoeConfig":
        _require(1 <= self.num_experts <= 256, "num_experts must be in [1, 256]")
        _require(1 <= self.num_experts_per_token <= 8, "num_experts_per_token must be in [1, 8]")
        _require(self.num_experts_per_token <= self.num_experts, "top-k exceeds expert count")
        _require(self.hidden_dim > 0 and self.intermediate_dim > 0, "dims must be positive")
        _require(self.capacity_factor > 0, "capacity_factor must be positive")
        return self


@dataclass
class FeedForwardType:
    """kind: 'dense' (up -> act -> down), 'gated' (SwiGLU) or 'moe'."""
    kind: str = "gated"
    intermediate_dim: int = 0
    activation: str = "silu"
    moe: Optional[MoeConfig] = None

    @staticmethod
    def dense(intermediate_dim: int, activation: str = "gelu") -> "FeedForwardType":
        return FeedForwardType("dense", intermediate_dim, activation)

    @staticmethod
    def gated(intermediate_dim: int) -> "FeedForwardType":
        return FeedForwardType("gated", intermediate_dim, "silu")

    @staticmethod
    def moe_(cfg: MoeConfig) -> "FeedForwardType":
        return FeedForwardType("moe", cfg.intermediate_dim, "silu", cfg)

    def validate(self) -> "FeedForwardType":
        _require(self.kind in ("dense", "gated", "moe"), f"unknown ff kind {self.kind}")
        if self.kind == "moe":
            _require(self.moe is not None, "moe ff needs a MoeConfig")
            self.moe.validate()
        else:
            _require(self.intermediate_dim > 0, "intermediate_dim must be positive")
        return self


@dataclass
class MlaConfig:
    num_heads: int
    head_dim: int            # non-rope part of the q/k head
    v_head_dim: int
    hidden_size: int
    kv_lora_rank: int
    q_lora_rank: int         # 0 = no q compression
    rope_head_dim: int
    rope_theta: float = 10000.0
    max_seq_len: int = 4096

    def validate(self) -> "MlaConfig":
        _require(self.num_heads > 0 and self.head_dim > 0 and self.v_head_dim > 0, "bad head dims")
        _require(self.kv_lora_rank > 0 and self.rope_head_dim % 2 == 0, "bad latent dims")
        return self


@dataclass
class TransformerConfig:
    hidden_size: int
    num_heads: int
    num_kv_heads: int
    head_dim: int
    num_layers: int
    vocab_size: int
    max_seq_len: int = 4096
    rope_theta: float = 10000.0
    rms_norm_eps: float = 1e-6
    ff_type: FeedForwardType = field(default_factory=FeedForwardType)
    rope_traditional: bool = False
    sliding_window: int = 0          # 0 = full attention
    tie_embeddings: bool = False
    first_dense_layers: int = 0      # DeepSeek: leading layers use a dense FFN
    dense_intermediate_dim: int = 0  # FFN width of those layers
    mla: Optional[MlaConfig] = None
    name: str = "transformer"

    def validate(self) -> "TransformerConfig":
        _require(self.hidden_size > 0 and self.num_layers > 0 and self.vocab_size > 0, "bad sizes")
        _require(self.num_heads > 0 and self.num_kv_heads > 0, "head counts must be positive")
        _require(self.num_kv_heads <= self.num_heads, "num_kv_heads must be <= num_heads")
        _require(self.num_heads % self.num_kv_heads == 0, "num_heads must be a multiple of num_kv_heads")
        _require(self.head_dim % 2 == 0, "head_dim must be even for RoPE")
        self.ff_type.validate()
        if self.mla is not None:
            self.mla.validate()
        return self

    @property
    def q_dim(self) -> int:
        return self.num_heads * self.head_dim

    @property
    def kv_dim(self) -> int:
        return self.num_kv_heads * self.head_dim

    def replace(self, **kw) -> "TransformerConfig":
        return dataclasses.replace(self, **kw)


@dataclass
class ScoredAttentionSpec:
    """Attention whose scores are modified before the softmax: ``scale``, a soft cap (0: none), and
    the per-head temperature, distance bias and sink that come with the weights. Query / key heads
    are ``dim`` wide, value heads ``vdim``."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float = 0.0

    def validate(self) -> "ScoredAttentionSpec":
        _require(self.heads > 0 and self.kv_heads > 0, "head counts must be positive")
        _require(self.heads % self.kv_heads == 0, "heads must be a multiple of kv_heads")
        _require(self.dim > 0 and self.vdim > 0, "head sizes must be positive")
        _require(self.softcap >= 0, "softcap must be >= 0 (0: no cap)")
        return self


@dataclass
class ParallelLayerSpec:
    """One layer of a parallel-block decoder: attention and (unless ``ff`` is 0) a dense feed-forward
    that read the same normalised input."""
    mixer: ScoredAttentionSpec
    ff: int = 0

    def validate(self) -> "ParallelLayerSpec":
        self.mixer.validate()
        _require(self.ff >= 0, "ff must be >= 0 (0: no feed-forward)")
        return self


@dataclass
class PosudraConfig:
    """Posudra: parallel-block decoder without rotation; every layer states its own sizes."""
    vocab_size: int
    width: int
    layers: "list[ParallelLayerSpec]"
    norm_eps: float = 1e-6
    embedding_scale: float = 1.0
    max_seq_len: int = 0             # 0: bounded by the cache only (positions enter as distances)
    name: str = "posudra"

    sliding_window = 0               # every key stays visible

    def validate(self) -> "PosudraConfig":
        _require(self.vocab_size > 0 and self.width > 0 and len(self.layers) > 0, "bad sizes")
        _require(self.norm_eps > 0, "norm_eps must be positive")
        for layer in self.layers:
            layer.validate()
        return self

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def hidden_size(self) -> int:
        return self.width

    @staticmethod
    def from_json(c: dict) -> "PosudraConfig":
        layers = []
        for i, e in enumerate(c["layers"]):
            _require(e.get("type") == "attention", f"layer {i}: unknown mixer type {e.get('type')!r}")
            m, mlp = e["mixer"], e.get("mlp")
            _require(mlp is None or mlp.get("kind") == "dense",
                     f"layer {i}: unknown feed-forward kind {None if mlp is None else mlp.get('kind')!r}")
            layers.append(ParallelLayerSpec(
                ScoredAttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]),
                                    float(m["scale"]), float(m.get("softcap") or 0.0)),
                0 if mlp is None else int(mlp["ff"])))
        return PosudraConfig(int(c["vocab"]), int(c["width"]), layers, float(c["norm"]["eps"]),
                             float(c["embedding"]["scale"])).validate()

    def to_json(self) -> dict:
        return {"architecture": "Posudra", "vocab": self.vocab_size, "width": self.width,
                "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embedding_scale},
                "layers": [{"type": "attention",
                            "mixer": {"heads": l.mixer.heads, "kv_heads": l.mixer.kv_heads, "dim": l.mixer.dim,
                                      "vdim": l.mixer.vdim, "scale": l.mixer.scale, "softcap": l.mixer.softcap},
                            "mlp": {"kind": "dense", "ff": l.ff} if l.ff else None} for l in self.layers]}


@dataclass
class WindowAttentionSpec:
    """Grouped-query attention without positions, per-head query / key norm, a sigmoid gate per head on
    the output and a sliding window (0: none)."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0

    kind = "attention"

    def validate(self) -> "WindowAttentionSpec":
        _require(self.heads > 0 and self.kv_heads > 0, "head counts must be positive")
        _require(self.heads % self.kv_heads == 0, "heads must be a multiple of kv_heads")
        _require(self.dim > 0 and self.vdim > 0, "head sizes must be positive")
        _require(self.window >= 0, "window must be >= 0 (0: none)")
        return self

    @staticmethod
    def from_json(m: dict) -> "WindowAttentionSpec":
        return WindowAttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                                   int((m.get("mask") or {}).get("size") or 0))

    def to_json(self) -> dict:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale,
                "mask": {"size": self.window} if self.window else None}


@dataclass
class LatentAttentionSpec:
    """Attention over one latent of ``kv_rank`` values and one rotated key part of ``rot_dim`` values per
    token; heads have ``dim`` unrotated and ``rot_dim`` rotated query / key values, of which the first
    ``rot_dims`` turn, and ``vdim`` value channels. ``q_rank``: queries go through a normed latent of that size (0:
    they do not). ``kv_from``: the layer whose cached latents and key parts this one reads (None: its own)."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot_base: float = 10000.0
    rot_dims: Optional[int] = None       # default: all of rot_dim
    q_rank: int = 0
    kv_from: Optional[int] = None

    kind = "latent_attention"

    def __post_init__(self):
        if self.rot_dims is None:
            self.rot_dims = self.rot_dim

    def validate(self) -> "LatentAttentionSpec":
        _require(self.heads > 0 and self.dim > 0 and self.vdim > 0 and self.kv_rank > 0, "sizes must be positive")
        _require(self.rot_dim >= 0 and self.rot_dims % 2 == 0 and self.rot_dims <= self.rot_dim,
                 "rotated dimensions come in pairs, at most rot_dim of them")
        _require(self.kv_rank <= 1024, "kv_rank must be <= 1024")
        _require(self.rot_base > 0, "rot_base must be positive")
        _require(self.q_rank >= 0, "q_rank must be >= 0 (0: no query latent)")
        return self

    @staticmethod
    def from_json(m: dict) -> "LatentAttentionSpec":
        rot = m.get("rot") or {}
        rot_dim = int(m["rot_dim"])
        return LatentAttentionSpec(int(m["heads"]), int(m["dim"]), rot_dim, int(m["vdim"]), int(m["kv_rank"]),
                                   float(m["scale"]), float(rot.get("base", 10000.0)), int(rot.get("dims", rot_dim)),
                                   int(m.get("q_rank") or 0), None if m.get("kv_from") is None else int(m["kv_from"]))

    def to_json(self) -> dict:
        out = {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "kv_rank": self.kv_rank,
               "scale": self.scale, "rot": {"base": self.rot_base, "dims": self.rot_dims}}
        if self.q_rank:
            out["q_rank"] = self.q_rank
        if self.kv_from is not None:
            out["kv_from"] = self.kv_from
        return out


@dataclass
class WkvSpec:
    """RWKV-style time mixing: ``heads`` states of dim x dim, decays from a low-rank projection (its
    rank comes with the weights; ``decay_rank`` is what random weights use)."""
    heads: int
    dim: int
    decay_rank: int = 16

    kind = "wkv"

    def validate(self) -> "WkvSpec":
        _require(self.heads > 0 and 0 < self.dim <= 256, "wkv: heads must be positive, dim in [1, 256]")
        return self

    @staticmethod
    def from_json(m: dict) -> "WkvSpec":
        return WkvSpec(int(m["heads"]), int(m["dim"]))

    def to_json(self) -> dict:
        return {"heads": self.heads, "dim": self.dim}


@dataclass
class ClampedFfSpec:
    """Gated feed-forward whose gate and up values are clamped to ``limit``."""
    ff: int
    limit: float

    def validate(self) -> "ClampedFfSpec":
        _require(self.ff > 0 and self.limit > 0, "feed-forward: ff and limit must be positive")
        return self

    def to_json(self) -> dict:
        return {"kind": "dense", "ff": self.ff, "limit": self.limit}


@dataclass
class RoutedFfSpec:
    """``experts`` clamped feed-forwards of width ``ff`` and ``identity`` experts that return their input;
    each token uses ``top`` of them, chosen by corrected softmax scores."""
    experts: int
    identity: int
    top: int
    ff: int
    limit: float

    def validate(self) -> "RoutedFfSpec":
        _require(self.experts > 0 and self.identity >= 0 and self.ff > 0 and self.limit > 0, "bad expert sizes")
        _require(self.experts <= 256 and self.experts + self.identity <= 512, "at most 256 experts and 512 router outputs")
        _require(1 <= self.top <= min(32, self.experts + self.identity), "top must be in [1, 32] and <= the router outputs")
        return self

    def to_json(self) -> dict:
        return {"kind": "moe", "expert": {"ff": self.ff, "limit": self.limit},
                "router": {"experts": self.experts, "identity": self.identity, "top": self.top}}


_MIXERS = {c.kind: c for c in (WindowAttentionSpec, LatentAttentionSpec, WkvSpec)}


@dataclass
class PostNormLayerSpec:
    """One layer: a mixer and (unless None) a feed-forward, each followed by a norm of its output."""
    mixer: "WindowAttentionSpec | LatentAttentionSpec | WkvSpec"
    mlp: "ClampedFfSpec | RoutedFfSpec | None" = None

    def validate(self) -> "PostNormLayerSpec":
        self.mixer.validate()
        if isinstance(self.mixer, LatentAttentionSpec):
            _require(not self.mixer.q_rank and self.mixer.kv_from is None, "latent attention: no query latent, no shared rows")
        if self.mlp is not None:
            self.mlp.validate()
        return self

    @staticmethod
    def from_json(e: dict) -> "PostNormLayerSpec":
        _require(e.get("type") in _MIXERS, f"unknown mixer type {e.get('type')!r}")
        m, mlp = e.get("mlp"), None
        if m is not None:
            _require(m.get("kind") in ("dense", "moe"), f"unknown feed-forward kind {m.get('kind')!r}")
            if m["kind"] == "dense":
                mlp = ClampedFfSpec(int(m["ff"]), float(m["limit"]))
            else:
                r, x = m["router"], m["expert"]
                mlp = RoutedFfSpec(int(r["experts"]), int(r.get("identity") or 0), int(r["top"]), int(x["ff"]),
                                   float(x["limit"]))
        return PostNormLayerSpec(_MIXERS[e["type"]].from_json(e["mixer"]), mlp)

    def to_json(self) -> dict:
        return {"type": self.mixer.kind, "mixer": self.mixer.to_json(),
                "mlp": None if self.mlp is None else self.mlp.to_json()}


@dataclass
class RodapelConfig:
    """Rodapel: a decoder that mixes windowed attention, latent attention and WKV recurrence, with norms on
    the sublayers' outputs; every layer states its own kind and sizes."""
    vocab_size: int
    width: int
    layers: "list[PostNormLayerSpec]"
    norm_eps: float = 1e-6
    max_seq_len: int = 0             # 0: bounded by the cache only
    name: str = "rodapel"

    sliding_window = 0               # pages are shared by every layer: none can be dropped early

    def validate(self) -> "RodapelConfig":
        _require(self.vocab_size > 0 and self.width > 0 and len(self.layers) > 0, "bad sizes")
        _require(self.norm_eps > 0, "norm_eps must be positive")
        for layer in self.layers:
            layer.validate()
        return self

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def hidden_size(self) -> int:
        return self.width

    @staticmethod
    def from_json(c: dict) -> "RodapelConfig":
        return RodapelConfig(int(c["vocab"]), int(c["width"]), [PostNormLayerSpec.from_json(e) for e in c["layers"]],
                             float(c["norm"]["eps"])).validate()

    def to_json(self) -> dict:
        return {"architecture": "Rodapel", "vocab": self.vocab_size, "width": self.width,
                "norm": {"eps": self.norm_eps}, "layers": [l.to_json() for l in self.layers]}


@dataclass
class RotarySpec:
    """Rotation of the first ``dims`` values of a head; ``scaling``: None, YaRN's (factor, original, fast, slow) or Llama's
    (factor, original, high, low)."""
    base: float
    dims: int
    scaling: Optional[dict] = None

    def validate(self, dim: int) -> "RotarySpec":
        _require(self.base > 0 and 0 <= self.dims <= dim and self.dims % 2 == 0,
                 "rotated dimensions come in pairs, at most the head's")
        if self.scaling:
            keys = self.scaling_keys(self.scaling)
            _require(all(float(self.scaling[k]) > 0 for k in keys), "rotation scaling: positive values")
            if "high" in keys:
                _require(self.scaling["high"] > self.scaling["low"], "rotation scaling: high must be above low")
            else:
                _require(self.base != 1.0, "rotation scaling needs a base other than 1")
        return self

    @staticmethod
    def scaling_keys(s: dict) -> tuple:
        return ("factor", "original", "high", "low") if "high" in s else ("factor", "original", "fast", "slow")

    @staticmethod
    def from_json(r: dict) -> "RotarySpec":
        s = r.get("scaling")
        return RotarySpec(float(r["base"]), int(r["dims"]),
                          None if not s else {k: float(s[k]) for k in RotarySpec.scaling_keys(s)})

    def to_json(self) -> dict:
        out = {"base": self.base, "dims": self.dims}
        if self.scaling:
            out["scaling"] = dict(self.scaling)
        return out


@dataclass
class ChunkedAttentionSpec:
    """Grouped-query attention with biased projections, rotated and unweightedly normed queries and keys, a soft cap
    (0: none) and, with ``chunk`` > 0, only the keys of the query's own chunk of so many positions."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: RotarySpec
    softcap: float = 0.0
    chunk: int = 0

    def validate(self) -> "ChunkedAttentionSpec":
        _require(self.heads > 0 and self.kv_heads > 0 and self.heads % self.kv_heads == 0,
                 "heads must be a positive multiple of kv_heads")
        _require(self.dim > 0 and self.vdim > 0, "head sizes must be positive")
        _require(self.softcap >= 0 and self.chunk >= 0, "softcap and chunk must be >= 0 (0: none)")
        self.rot.validate(self.dim)
        return self

    @staticmethod
    def from_json(m: dict) -> "ChunkedAttentionSpec":
        return ChunkedAttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                                    RotarySpec.from_json(m["rot"]), float(m.get("softcap") or 0.0),
                                    int((m.get("mask") or {}).get("size") or 0))

    def to_json(self) -> dict:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale,
                "rot": self.rot.to_json(), "softcap": self.softcap or None, "mask": {"size": self.chunk} if self.chunk else None}


@dataclass
class StateSpaceSpec:
    """State-space heads: ``heads`` states of ``state`` x ``vdim``, ``groups`` shared input / output vectors, a causal
    convolution over ``conv`` tokens, the gated output normed in ``norm_groups`` equal parts."""
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        return self.inner + 2 * self.groups * self.state

    def validate(self) -> "StateSpaceSpec":
        _require(self.heads > 0 and self.vdim > 0 and 0 < self.state <= 256, "state space: heads and vdim positive, state in [1, 256]")
        _require(self.groups > 0 and self.heads % self.groups == 0, "state space: heads must be a multiple of groups")
        _require(self.conv > 0, "state space: the convolution has at least one tap")
        _require(self.norm_groups > 0 and self.inner % self.norm_groups == 0, "state space: norm groups must divide the inner width")
        return self

    @staticmethod
    def from_json(m: dict) -> "StateSpaceSpec":
        return StateSpaceSpec(*(int(m[k]) for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups")))

    def to_json(self) -> dict:
        return {k: getattr(self, k) for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups")}


@dataclass
class GlaSpec:
    """Gated linear attention: ``heads`` states of ``dim`` x ``vdim``, decays sigmoid(z)^(1 / tau) from a low-rank
    projection (its rank comes with the weights; ``decay_rank`` is what random weights use)."""
    heads: int
    dim: int
    vdim: int
    tau: float
    decay_rank: int = 16

    kind = "gla"

    def validate(self) -> "GlaSpec":
        _require(self.heads > 0 and self.vdim > 0 and 0 < self.dim <= 256, "gla: heads and vdim positive, dim in [1, 256]")
        _require(self.tau > 0, "gla: tau must be positive")
        return self

    @staticmethod
    def from_json(m: dict) -> "GlaSpec":
        return GlaSpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["tau"]))

    def to_json(self) -> dict:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "tau": self.tau}


@dataclass
class PairSpec:
    """Chunked attention and state-space heads side by side on the same input, their outputs weighted."""
    left: ChunkedAttentionSpec
    right: StateSpaceSpec
    left_scale: float = 1.0
    right_scale: float = 1.0

    kind = "parallel"

    def validate(self) -> "PairSpec":
        self.left.validate()
        self.right.validate()
        return self

    @staticmethod
    def from_json(m: dict) -> "PairSpec":
        return PairSpec(ChunkedAttentionSpec.from_json(m["left"]), StateSpaceSpec.from_json(m["right"]),
                        float(m["left_scale"]), float(m["right_scale"]))

    def to_json(self) -> dict:
        return {"left": self.left.to_json(), "right": self.right.to_json(), "left_scale": self.left_scale,
                "right_scale": self.right_scale}


@dataclass
class SwigluFfSpec:
    """Gated feed-forward with silu."""
    ff: int

    limit = 0.0                      # of the gated activation: none

    def validate(self) -> "SwigluFfSpec":
        _require(self.ff > 0, "feed-forward: ff must be positive")
        return self

    def to_json(self) -> dict:
        return {"kind": "dense", "ff": self.ff}


@dataclass
class ChosenFfSpec:
    """``experts`` gated feed-forwards of width ``ff``; each token uses the ``top`` with the largest biased logits,
    weighted by the softmax over those alone."""
    experts: int
    top: int
    ff: int

    limit = 0.0
    identity = 0

    def validate(self) -> "ChosenFfSpec":
        _require(0 < self.experts <= 256 and self.ff > 0, "experts: 1 to 256, ff positive")
        _require(1 <= self.top <= min(32, self.experts), "top must be in [1, 32] and <= experts")
        return self

    def to_json(self) -> dict:
        return {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top}}


_TWIN_MIXERS = {c.kind: c for c in (LatentAttentionSpec, GlaSpec, PairSpec)}


@dataclass
class TwinNormLayerSpec:
    """One layer: a mixer and (unless None) a feed-forward, both reading the same residual through norms of their own."""
    mixer: "LatentAttentionSpec | GlaSpec | PairSpec"
    mlp: "SwigluFfSpec | ChosenFfSpec | None" = None

    def validate(self) -> "TwinNormLayerSpec":
        self.mixer.validate()
        if isinstance(self.mixer, LatentAttentionSpec):
            _require(self.mixer.q_rank > 0, "latent attention: queries go through a latent (q_rank)")
        if self.mlp is not None:
            self.mlp.validate()
        return self

    @staticmethod
    def from_json(e: dict) -> "TwinNormLayerSpec":
        _require(e.get("type") in _TWIN_MIXERS, f"unknown mixer type {e.get('type')!r}")
        m, mlp = e.get("mlp"), None
        if m is not None:
            _require(m.get("kind") in ("dense", "moe"), f"unknown feed-forward kind {m.get('kind')!r}")
            mlp = SwigluFfSpec(int(m["ff"])) if m["kind"] == "dense" else \
                ChosenFfSpec(int(m["router"]["experts"]), int(m["router"]["top"]), int(m["expert"]["ff"]))
        return TwinNormLayerSpec(_TWIN_MIXERS[e["type"]].from_json(e["mixer"]), mlp)

    def to_json(self) -> dict:
        return {"type": self.mixer.kind, "mixer": self.mixer.to_json(),
                "mlp": None if self.mlp is None else self.mlp.to_json()}


@dataclass
class NugosunConfig:
    """Nugosun: a decoder of latent attention (rows may be shared between layers), gated linear attention and pairs of
    chunked attention and state-space heads, with the feed-forward beside the mixer; every layer states its own kind
    and sizes."""
    vocab_size: int
    width: int
    layers: "list[TwinNormLayerSpec]"
    norm_eps: float = 1e-6
    embedding_scale: float = 1.0
    max_seq_len: int = 0             # 0: bounded by the cache only
    name: str = "nugosun"

    sliding_window = 0               # pages are shared by every layer: none can be dropped early

    def validate(self) -> "NugosunConfig":
        _require(self.vocab_size > 0 and self.width > 0 and len(self.layers) > 0, "bad sizes")
        _require(self.norm_eps > 0, "norm_eps must be positive")
        for i, layer in enumerate(self.layers):
            layer.validate()
            j = getattr(layer.mixer, "kv_from", None)
            if j is not None:
                _require(0 <= j < i and isinstance(self.layers[j].mixer, LatentAttentionSpec), f"layer {i}: kv_from names no latent layer before it")
                a, b = layer.mixer, self.layers[j].mixer
                _require(b.kv_from is None, f"layer {i}: kv_from names a layer without rows of its own")
                _require((a.kv_rank, a.rot_dim, a.rot_dims, a.rot_base) == (b.kv_rank, b.rot_dim, b.rot_dims, b.rot_base),
                         f"layer {i}: the shared rows' sizes and rotation differ")
        return self

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def hidden_size(self) -> int:
        return self.width

    @staticmethod
    def from_json(c: dict) -> "NugosunConfig":
        return NugosunConfig(int(c["vocab"]), int(c["width"]), [TwinNormLayerSpec.from_json(e) for e in c["layers"]],
                             float(c["norm"]["eps"]), float(c["embedding"]["scale"])).validate()

    def to_json(self) -> dict:
        return {"architecture": "Nugosun", "vocab": self.vocab_size, "width": self.width, "norm": {"eps": self.norm_eps},
                "embedding": {"scale": self.embedding_scale}, "layers": [l.to_json() for l in self.layers]}


@dataclass
class DifferentialAttentionSpec:
    """Grouped-query attention with two maps per head (a query and a key of ``dim`` values each, over the same values): the
    first map's result minus a learned multiple of the second's, normed per head and times 1 - ``diff``. Neighbouring values
    of queries and keys turn together; ``window`` > 0: only the last so many keys."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: RotarySpec
    diff: float
    window: int = 0

    kind = "attention"

    def validate(self) -> "DifferentialAttentionSpec":
        _require(self.heads > 0 and self.kv_heads > 0 and self.heads % self.kv_heads == 0,
                 "heads must be a positive multiple of kv_heads")
        _require(self.dim > 0 and self.vdim > 0, "head sizes must be positive")
        _require(self.window >= 0, "window must be >= 0 (0: none)")
        self.rot.validate(self.dim)
        return self

    @staticmethod
    def from_json(m: dict) -> "DifferentialAttentionSpec":
        return DifferentialAttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                                         RotarySpec.from_json(m["rot"]) if m.get("rot") else RotarySpec(10000.0, 0),
                                         float(m["diff"]), int((m.get("mask") or {}).get("size") or 0))

    def to_json(self) -> dict:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale,
                "rot": self.rot.to_json(), "diff": self.diff, "mask": {"size": self.window} if self.window else None}


@dataclass
class LightningSpec:
    """Lightning attention: ``heads`` states of ``dim`` x ``vdim``, each with a constant decay."""
    heads: int
    dim: int
    vdim: int
    decay: "list[float]"

    kind = "lightning"

    def validate(self) -> "LightningSpec":
        _require(self.heads > 0 and self.vdim > 0 and 0 < self.dim <= 256, "lightning: heads and vdim positive, dim in [1, 256]")
        _require(len(self.decay) == self.heads, "lightning: one decay per head")
        return self

    @staticmethod
    def from_json(m: dict) -> "LightningSpec":
        return LightningSpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]), [float(v) for v in m["decay"]])

    def to_json(self) -> dict:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}


@dataclass
class PolyNormFfSpec:
    """Feed-forward without a gate, its activation a polynomial of normed powers."""
    ff: int

    def validate(self) -> "PolyNormFfSpec":
        _require(self.ff > 0, "feed-forward: ff must be positive")
        return self

    def to_json(self) -> dict:
        return {"kind": "dense", "ff": self.ff}


@dataclass
class GroupedFfSpec:
    """``experts`` gated feed-forwards of width ``ff`` in ``groups`` equal groups; each token uses the ``top`` with the largest
    sigmoid scores in its ``keep`` best groups, weighted by the scores times ``scale``, and (``shared`` > 0) one of width
    ``shared`` that every token uses."""
    experts: int
    top: int
    ff: int
    groups: int = 1
    keep: int = 1
    scale: float = 1.0
    shared: int = 0

    limit = 0.0
    identity = 0

    def validate(self) -> "GroupedFfSpec":
        _require(0 < self.experts <= 256 and self.ff > 0 and self.shared >= 0, "experts: 1 to 256, ff positive")
        _require(1 <= self.groups <= 128 and self.experts % self.groups == 0 and 1 <= self.keep <= self.groups,
                 "experts must form 1 to 128 equal groups, of which 1 or more are kept")
        _require(1 <= self.top <= min(31, self.keep * self.experts // self.groups), "top must be in [1, 31] and fit the kept groups")
        return self

    @property
    def slices(self) -> tuple:
        """(count, width) of the equal parts the shared feed-forward is cut into, which run as experts of every token, as wide
        as the routed ones unless they would be too many."""
        if not self.shared:
            return 0, self.ff
        n = min(-(-self.shared // self.ff), 32 - self.top, 512 - self.experts)
        return n, max(self.ff, -(-self.shared // n))

    def to_json(self) -> dict:
        out = {"kind": "moe", "expert": {"ff": self.ff},
               "router": {"experts": self.experts, "top": self.top, "scale": self.scale, "groups": {"count": self.groups, "keep": self.keep}}}
        if self.shared:
            out["shared"] = {"ff": self.shared}
        return out


_SANDWICH_MIXERS = {c.kind: c for c in (DifferentialAttentionSpec, LightningSpec)}


@dataclass
class SandwichLayerSpec:
    """One layer: a mixer and (unless None) a feed-forward, each between two norms and behind a short convolution."""
    mixer: "DifferentialAttentionSpec | LightningSpec"
    mlp: "PolyNormFfSpec | GroupedFfSpec | None" = None

    def validate(self) -> "SandwichLayerSpec":
        self.mixer.validate()
        if self.mlp is not None:
            self.mlp.validate()
        return self

    @staticmethod
    def from_json(e: dict) -> "SandwichLayerSpec":
        _require(e.get("type") in _SANDWICH_MIXERS, f"unknown mixer type {e.get('type')!r}")
        m, mlp = e.get("mlp"), None
        if m is not None:
            _require(m.get("kind") in ("dense", "moe"), f"unknown feed-forward kind {m.get('kind')!r}")
            if m["kind"] == "dense":
                mlp = PolyNormFfSpec(int(m["ff"]))
            else:
                r, g = m["router"], m["router"].get("groups") or {}
                mlp = GroupedFfSpec(int(r["experts"]), int(r["top"]), int(m["expert"]["ff"]), int(g.get("count", 1)),
                                    int(g.get("keep", 1)), float(r.get("scale", 1.0)), int((m.get("shared") or {}).get("ff", 0)))
        return SandwichLayerSpec(_SANDWICH_MIXERS[e["type"]].from_json(e["mixer"]), mlp)

    def to_json(self) -> dict:
        return {"type": self.mixer.kind, "mixer": self.mixer.to_json(),
                "mlp": None if self.mlp is None else self.mlp.to_json()}


@dataclass
class LoopSpec:
    """Layers ``start`` .. ``stop`` - 1 run ``times`` times in a row, each pass with a cache of its own."""
    start: int
    stop: int
    times: int

    def validate(self, layers: int) -> "LoopSpec":
        _require(0 <= self.start < self.stop <= layers and self.times >= 1, "loop: a range of layers, at least once")
        return self


@dataclass
class NizoraxConfig:
    """Nizorax: a decoder of differential attention and lightning attention between layer norms, with short convolutions over
    what the sublayers read and a range of layers that runs several times; every layer states its own kind and sizes."""
    vocab_size: int
    width: int
    layers: "list[SandwichLayerSpec]"
    norm_eps: float = 1e-6
    embedding_scale: float = 1.0
    logit_scale: float = 1.0
    taps: int = 4
    loop: Optional[LoopSpec] = None
    max_seq_len: int = 0             # 0: bounded by the cache only
    name: str = "nizorax"

    sliding_window = 0               # pages are shared by every layer: none can be dropped early

    def validate(self) -> "NizoraxConfig":
        _require(self.vocab_size > 0 and self.width > 0 and len(self.layers) > 0, "bad sizes")
        _require(self.norm_eps > 0, "norm_eps must be positive")
        _require(1 <= self.taps <= 64, "the short convolution has 1 to 64 taps")
        for layer in self.layers:
            layer.validate()
        if self.loop is not None:
            self.loop.validate(len(self.layers))
        return self

    @property
    def runs(self) -> "list[int]":
        """The layers in the order in which they run."""
        order = list(range(len(self.layers)))
        if self.loop is None:
            return order
        a, b = self.loop.start, self.loop.stop
        return order[:a] + order[a:b] * self.loop.times + order[b:]

    @property
    def num_layers(self) -> int:
        """Layer runs: what the cache holds pages and states for."""
        return len(self.runs)

    @property
    def hidden_size(self) -> int:
        return self.width

    @staticmethod
    def from_json(c: dict) -> "NizoraxConfig":
        loop = c.get("loop")
        return NizoraxConfig(int(c["vocab"]), int(c["width"]), [SandwichLayerSpec.from_json(e) for e in c["layers"]],
                             float(c["norm"]["eps"]), float((c.get("embedding") or {}).get("scale", 1.0)),
                             float(c.get("logit_scale", 1.0)), int(c["canon"]["taps"]),
                             LoopSpec(int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else None).validate()

    def to_json(self) -> dict:
        out = {"architecture": "Nizorax", "vocab": self.vocab_size, "width": self.width, "norm": {"eps": self.norm_eps},
               "embedding": {"scale": self.embedding_scale}, "logit_scale": self.logit_scale, "canon": {"taps": self.taps},
               "layers": [l.to_json() for l in self.layers]}
        if self.loop is not None:
            out["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        return out


@dataclass
class AttentionConfig:
    num_heads: int
    num_kv_heads: int
    head_dim: int
    max_seq_len: int = 4096
    rope_theta: float = 10000.0

    def validate(self) -> "AttentionConfig":
        _require(self.num_heads % self.num_kv_heads == 0, "heads must divide by kv heads")
        return self


@dataclass
class RotaryConfig:
    head_dim: int
    max_seq_len: int
    base_freq: float = 10000.0
    scale: float = 1.0
    traditional: bool = False


@dataclass
class QuantConfig:
    """MLX affine weight-only quantisation: w = scale * q + bias per group."""
    bits: int = 4
    group_size: int = 64

    def validate(self) -> "QuantConfig":
        _require(self.bits in (2, 3, 4, 6, 8), "bits must be one of 2,3,4,6,8")
        _require(self.group_size in (32, 64, 128), "group_size must be 32, 64 or 128")
        return self


@dataclass
class SchedulerConfig:
    max_batch_size: int = 64
    eos_token_id: int = -1
    block_size: int = 16
    max_prefill_chunk: int = 512

    def validate(self) -> "SchedulerConfig":
        _require(self.max_batch_size > 0 and self.block_size > 0, "bad scheduler sizes")
        _require(self.max_prefill_chunk > 0, "max_prefill_chunk must be positive")
        return self


@dataclass
class SamplerConfig:
    temperature: float = 0.0        # 0 = greedy
    top_k: int = 0                  # 0 = off
    top_p: float = 1.0              # 1 = off
    repetition_penalty: float = 1.0 # 1 = off
    seed: Optional[int] = None

    def validate(self) -> "SamplerConfig":
        _require(self.temperature >= 0, "temperature must be >= 0")
        _require(0 < self.top_p <= 1.0, "top_p must be in (0, 1]")
        _require(self.top_k >= 0, "top_k must be >= 0")
        _require(self.repetition_penalty > 0, "repetition_penalty must be > 0")
        return self


@dataclass
class InitConfig:
    """Process-group bring-up. Resolution order for rank/world: explicit fields, then RMLX_* env,
    then torchrun (RANK/WORLD_SIZE), then OMPI/PMI/SLURM env, else (0, 1)."""
    rank: Optional[int] = None
    world_size: Optional[int] = None
    backend: str = "auto"           # auto | nccl | gloo | loopback
    strict: bool = False            # fail instead of falling back to loopback
    master_addr: str = "127.0.0.1"
    master_port: int = 18520
    timeout_s: float = 120.0


# ------------------------------------------------------------------------------------------------
# Presets
# ------------------------------------------------------------------------------------------------
def tiny_dense_config() -> TransformerConfig:
    """The CPU plumbing config: hidden 256, 4 q / 2 kv heads, head_dim 64, SwiGLU 688, vocab 1024."""
    return TransformerConfig(hidden_size=256, num_heads=4, num_kv_heads=2, head_dim=64, num_layers=2,
                             vocab_size=1024, max_seq_len=256, rope_theta=1e4, rms_norm_eps=1e-6,
                             ff_type=FeedForwardType.gated(688), name="tiny-dense").validate()


def moe_a22b_config(num_layers: int = 60, max_seq_len: int = 8192) -> TransformerConfig:
    """MoE-A22B-shaped decoder: hidden 4096, 64 q / 4 kv heads, head_dim 128, theta 1e6, 128 experts
    top-8 with expert SwiGLU width 1536, vocab 151936."""
    moe = MoeConfig(num_experts=128, num_experts_per_token=8, hidden_dim=4096, intermediate_dim=1536)
    return TransformerConfig(hidden_size=4096, num_heads=64, num_kv_heads=4, head_dim=128,
                             num_layers=num_layers, vocab_size=151936, max_seq_len=max_seq_len,
                             rope_theta=1e6, rms_norm_eps=1e-6, ff_type=FeedForwardType.moe_(moe),
                             name="moe-a22b").validate()
