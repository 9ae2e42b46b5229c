"""What models with a layer list of their own share (``models/rodapel.py``, ``models/nugosun.py``, ``models/nizorax.py``): merged and padded
weights, activation buffers, latent attention over the paged cache, gated and routed feed-forwards, and the forward
pass over a ragged batch with its one-sequence conveniences. A model adds its mixers, ``start`` (embedding) and
``layer``."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Dict, List, Optional, Sequence, Tuple

import torch

from .. import _lib
from ..config import LatentAttentionSpec
from ..kv.paged import PAGE, PagedKvCache
from ..ops import latent as L
from ..ops import parallel_block as P
from ..ops import post_norm as N
from ..ops import routed as R
from ..ops import twin_norm as TN
from ..ops.decode import default_splits
from ..ops.gemm import GemmStatus
from ..ops.parallel_block import ScoreMods, pad8
from ..ops.post_norm import pad_to
from ..ops.weights import LinearWeight, W_BF16
from .ragged import Entry, RaggedBatch

# Latent attention: batch entries of up to this many tokens attend to the cached latents; longer ones to keys
# and values expanded for their whole context (which costs about as much as 0.8 * kv_rank query tokens).
LATENT_ABSORB = 4
LATENT_ROW_PAD = 8       # unused values behind a latent cache row (csrc/kernels/mla_decode.cu)


# ------------------------------------------------------------------------------------------------
# Weights
# ------------------------------------------------------------------------------------------------
@dataclass
class LatentWeights:
    spec: LatentAttentionSpec
    source: int                      # the layer whose cache rows are read
    w_in: LinearWeight               # [rows, width_p]: q (or the query latent) | latent | rotated key part
    down_at: int                     # column of the latent in a row of w_in's result
    q_norm: Optional[torch.Tensor]   # fp32 [pad8(q_rank)]; None: no query latent
    w_uq: Optional[LinearWeight]     # [rows, pad8(q_rank)]
    c_norm: Optional[torch.Tensor]   # fp32 [rank]; None: the rows are another layer's
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
class DenseFfWeights:
    spec: object                     # ff and limit of the gated activation
    w_gu: LinearWeight               # [2 * ff_p, width_p]: gate | up
    w_down: LinearWeight             # [width_p, ff_p]


@dataclass
class RoutedFfWeights:
    spec: object                     # experts, identity, top, ff, limit
    router: torch.Tensor             # [experts + identity, width_p]
    correction: Optional[torch.Tensor]   # fp32 [experts + identity]: the router's correction or bias (None: neither)
    w_gu: LinearWeight               # [experts + always, 2 * ff_p, width_p]
    w_down: LinearWeight             # [experts + always, rows, ff_p], rows: width rounded up to the tile width
    always: int = 0                  # experts behind the routed ones that every token uses


def weight_bytes(*parts) -> int:
    """Bytes of the tensors and linear weights that the given dataclasses hold (one given twice counts once)."""
    def size(v) -> int:
        if isinstance(v, LinearWeight):
            return v.nbytes()
        return v.numel() * v.element_size() if isinstance(v, torch.Tensor) else 0
    return sum(size(v) for p in {id(p): p for p in parts if p is not None}.values() for v in vars(p).values())


def check_tensors(tensors: Dict[str, torch.Tensor], shapes: Dict[str, tuple]) -> None:
    for name, shape in shapes.items():
        if name not in tensors:
            raise KeyError(f"checkpoint has no tensor {name!r}")
        if tuple(tensors[name].shape) != shape:
            raise ValueError(f"{name}: shape {tuple(tensors[name].shape)}, expected {shape}")


class WeightBuilder:
    """Runtime weights from checkpoint tensors: projections merged and zero-padded, per-channel vectors in fp32."""

    def __init__(self, tensors: Dict[str, torch.Tensor], width: int, device, dtype):
        self.tensors, self.width, self.width_p, self.device, self.dtype = tensors, width, pad8(width), device, dtype

    def dev(self, t: torch.Tensor) -> torch.Tensor:
        return t.to(device=self.device, dtype=self.dtype)

    def zeros(self, *shape: int) -> torch.Tensor:
        return torch.zeros(*shape, dtype=self.dtype, device=self.device)

    def mat(self, parts, rows: int, cols: int) -> torch.Tensor:
        """Stack ``parts`` into a zero-padded [rows, cols] matrix."""
        out, at = self.zeros(rows, cols), 0
        for t in parts:
            out[at:at + t.shape[0], :t.shape[1]] = self.dev(t)
            at += t.shape[0]
        return out

    def lin(self, parts, rows: int, cols: int) -> LinearWeight:
        return LinearWeight(W_BF16, self.mat(parts, rows, cols))

    def vec(self, t: torch.Tensor, n: Optional[int] = None) -> torch.Tensor:
        out = torch.zeros(n or t.numel(), dtype=torch.float32, device=self.device)
        out[:t.numel()] = t.reshape(-1).to(device=self.device, dtype=torch.float32)
        return out

    def out_proj(self, t: torch.Tensor, heads: int, vdim: int) -> LinearWeight:
        """Attention writes heads at stride pad8(vdim): the projection's columns are spread likewise."""
        wo = self.zeros(self.width_p, heads, pad8(vdim))
        wo[:self.width, :, :vdim] = self.dev(t).view(self.width, heads, vdim)
        return LinearWeight(W_BF16, wo.view(self.width_p, -1))

    def latent(self, p: str, i: int, m: LatentAttentionSpec) -> LatentWeights:
        """Latent attention under the tensor prefix ``p`` (layer ``i``)."""
        g = lambda n: self.tensors[p + n]                                # noqa: E731
        q_cols = m.heads * (m.dim + m.rot_dim)
        own = m.kv_from is None
        down = [g("dkv")] if own else []
        q_norm = w_uq = None
        if m.q_rank:
            first, down_at = g("dq"), pad8(m.q_rank)
            q_norm, w_uq = self.vec(g("dq.norm"), down_at), self.lin([g("uq")], pad8(q_cols), pad8(m.q_rank))
        else:
            first, down_at = g("q"), q_cols
        rows = down_at + (m.kv_rank + m.rot_dim if own else 0)
        w_in = self.mat([self.mat([first], down_at, self.width_p)] + down, pad8(rows), self.width_p)
        uk = self.zeros(m.heads, pad8(m.kv_rank), pad8(m.dim))
        uk[:, :m.kv_rank, :m.dim] = self.dev(g("uk")).view(m.heads, m.dim, m.kv_rank).transpose(1, 2)
        uv = self.zeros(m.heads, pad8(m.vdim), pad8(m.kv_rank))
        uv[:, :m.vdim, :m.kv_rank] = self.dev(g("uv")).view(m.heads, m.vdim, m.kv_rank)
        ukv = torch.cat([uk.transpose(1, 2), uv], 1).reshape(-1, pad8(m.kv_rank)).contiguous()
        return LatentWeights(m, i if own else m.kv_from, LinearWeight(W_BF16, w_in), down_at, q_norm, w_uq,
                             self.vec(g("dkv.norm")) if own else None, uk, uv, LinearWeight(W_BF16, ukv),
                             self.out_proj(g("o"), m.heads, m.vdim),
                             self.vec(TN.rotary_frequencies(m.rot_base, m.rot_dims)[0]), ScoreMods(m.scale))

    def _gate_up(self, p: str, f, out: torch.Tensor, ffp: int) -> None:
        out[:f.ff, :self.width], out[ffp:ffp + f.ff, :self.width] = self.dev(self.tensors[p + "gate"]), self.dev(self.tensors[p + "up"])

    def dense(self, p: str, f) -> DenseFfWeights:
        ffp = pad_to(f.ff, 64)
        gu = self.zeros(2 * ffp, self.width_p)
        self._gate_up(p, f, gu, ffp)
        return DenseFfWeights(f, LinearWeight(W_BF16, gu), self.lin([self.tensors[p + "down"]], self.width_p, ffp))

    def routed(self, p: str, f, correction: str) -> RoutedFfWeights:
        ffp = pad_to(f.ff, 64)
        gu = self.zeros(f.experts, 2 * ffp, self.width_p)
        down = self.zeros(f.experts, pad_to(self.width_p, 128), ffp)
        for e in range(f.experts):
            self._gate_up(f"{p}e{e}.", f, gu[e], ffp)
            down[e, :self.width, :f.ff] = self.dev(self.tensors[f"{p}e{e}.down"])
        return RoutedFfWeights(f, self.mat([self.tensors[p + "router"]], f.experts + f.identity, self.width_p),
                               self.vec(self.tensors[p + correction]), LinearWeight(W_BF16, gu), LinearWeight(W_BF16, down))


def latent_row(m: LatentAttentionSpec) -> Optional[tuple]:
    """(kv heads, key row, value row) of a latent layer's pages: rows are key and value at once. None: the rows are
    another layer's."""
    return None if m.kv_from is not None else (1, pad8(m.kv_rank) + pad8(m.rot_dim) + LATENT_ROW_PAD, 0)


def save_checkpoint(model_dir: str, cfg, tensors: Dict[str, torch.Tensor]) -> None:
    """config.json and model.safetensors of a model."""
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


class RaggedModel:
    """One GPU's weights and the forward passes over them. ``kv_shapes`` / ``state_shapes``: what the cache holds per
    layer; ``min_heads``: query heads of the narrowest attention layer (plans the prompt tiles)."""

    # a step may hold prompt portions and decoded tokens together (``forward_batch``)
    mixed_batches = True
    title = "this model"

    def __init__(self, weights, kv_shapes: List[Optional[tuple]], state_shapes: List[Optional[Dict[str, tuple]]],
                 min_heads: int):
        self.w, self.cfg, self.layout = weights, weights.cfg, weights.layout
        self.device = weights.embed.device
        self.dtype = weights.embed.dtype
        self.width_p = pad8(self.cfg.width)
        self.allgather_logits = None
        self._kv_shapes, self._state_shapes, self._min_heads = kv_shapes, state_shapes, min_heads
        self._bufs: Optional[Buffers] = None
        self._scratch: Dict[tuple, object] = {}
        latent = [l.mix for l in weights.layers if isinstance(l.mix, LatentWeights)]
        self._absorb = LATENT_ABSORB if self.device.type == "cuda" and any(map(self.latent_prefill, latent)) else None

    @classmethod
    def from_checkpoint(cls, model_dir: str, device="cuda", dtype=torch.bfloat16):
        from .registry import from_pretrained
        return from_pretrained(model_dir, device, dtype)

    # ------------------------------------------------------------------ of the model
    def start(self, tokens: torch.Tensor, bufs: Buffers, pdl: bool = False) -> Tuple[torch.Tensor, ...]:
        """The activations that ``layer`` takes, for the tokens; the fp32 residual first."""
        raise NotImplementedError

    def layer(self, li: int, acts: Tuple[torch.Tensor, ...], c: StepContext) -> None:
        raise NotImplementedError

    # ------------------------------------------------------------------ cache
    def new_cache(self, num_blocks: int, max_seqs: int = 64, max_blocks_per_seq: Optional[int] = None,
                  dtype=None, kv_quant: Optional[str] = None) -> PagedKvCache:
        """``num_blocks`` pages of 16 tokens (page 0 is reserved). Without ``max_blocks_per_seq`` one
        sequence may take the whole pool, or ``cfg.max_seq_len`` tokens if that is set."""
        if kv_quant is not None:
            raise ValueError(f"{self.title}'s attention kernels read 16- or 32-bit caches")
        if max_blocks_per_seq is None:
            max_blocks_per_seq = max(1, num_blocks - 1)
            if self.cfg.max_seq_len:
                max_blocks_per_seq = min(max_blocks_per_seq, (self.cfg.max_seq_len + PAGE - 1) // PAGE)
        shapes = self._kv_shapes
        first = next((s for s in shapes if s is not None), (1, 8, 8))
        return PagedKvCache(num_blocks, len(shapes), first[0], first[1], dtype=dtype or self.dtype, device=self.device,
                            max_seqs=max_seqs, max_blocks_per_seq=max_blocks_per_seq, layer_shapes=shapes,
                            layer_states=self._state_shapes)

    # ------------------------------------------------------------------ attention
    def scratch(self, heads: int, kv_heads: int, vdim_p: int, rows: int, splits: int) -> P.ScoredDecodeScratch:
        """Split-KV scratch, shared by every layer of the same head shape."""
        key = (heads, kv_heads, vdim_p, rows, splits)
        if key not in self._scratch:
            self._scratch[key] = P.ScoredDecodeScratch(rows, heads, kv_heads, vdim_p, splits, self.device)
        return self._scratch[key]

    def attention_splits(self, m, rows: int, max_len: int, reach: int = 0) -> int:
        """KV splits of decode attention; ``reach`` > 0: a query sees at most so many keys."""
        if reach:
            max_len = min(max_len, reach + PAGE)
        return default_splits(rows, m.kv_heads, (m.heads // m.kv_heads + 15) // 16, max_len)

    def tensor_core_attention(self, m) -> bool:
        return self.dtype == torch.bfloat16 and P.decode_scored_supported(pad8(m.dim), pad8(m.vdim)) and \
            P.prefill_scored_supported(pad8(m.dim), pad8(m.vdim))

    def paged_attention(self, li: int, m, mods: ScoreMods, q: torch.Tensor, c: StepContext, window: int = 0, chunk: int = 0,
                        gate: Optional[torch.Tensor] = None, diff: Optional[P.MapDiff] = None) -> torch.Tensor:
        """Attention of the batch's queries [T, heads, pad8(dim)] over the layer's pages: tensor-core prompt attention for
        the entries of several tokens, split-KV decode attention for the others. ``diff``: differential attention, queries
        [T, heads, 2, pad8(dim)]; the batch's query tiles are then planned one lane wide."""
        t, b, pdl = c.t, c.batch, c.pdl
        k, v = c.cache.k[li], c.cache.v[li]
        attn = c.bufs.get("attn", t, m.heads, v.shape[3], dtype=self.dtype)
        see = dict(window=window, chunk=chunk, gate=gate)
        reach = min([r for r in (window, chunk) if r], default=0)
        rows_per_head = 1 if diff is None else 2
        if not self.tensor_core_attention(m):
            P.attention_any(q, k, v, c.block_table, c.positions, c.token_seq, mods, attn, diff=diff, vdim=m.vdim, pdl=pdl, **see)
        elif b is None:
            s = self.scratch(m.heads * rows_per_head, m.kv_heads, v.shape[3], t, self.attention_splits(m, t, c.max_len, reach))
            P.flash_decode_scored(k, v, c.block_table, c.positions, mods, attn, s, m.heads, m.dim, m.vdim, q=q, n_rows=t,
                                  diff=diff, pdl=pdl, **see)
        else:
            if b.tiles is not None and diff is not None:
                P.flash_prefill_diff(q, k, v, c.block_table, b.tiles, mods.scale, diff, m.vdim, attn, window=window, chunk=chunk)
            elif b.tiles is not None:
                P.flash_prefill_scored(q, k, v, c.block_table, b.tiles, mods, attn, lanes=b.lanes, **see)
            if b.single is not None:
                n = len(b.single_host)
                s = self.scratch(m.heads * rows_per_head, m.kv_heads, v.shape[3], n, self.attention_splits(m, n, b.single_len, reach))
                P.flash_decode_scored(k, v, c.block_table, c.positions, mods, attn, s, m.heads, m.dim, m.vdim, q=q,
                                      rows=b.single, table_rows=c.token_seq, diff=diff, **see)
        return attn.view(t, -1)

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
        """Everything between the two projections: raw [T, q or its latent | latent | key part] -> attention output rows."""
        m, t, dt, pdl = mw.spec, c.t, self.dtype, c.pdl
        pool, b = c.cache.k[mw.source], c.batch
        q_raw = raw
        if mw.w_uq is not None:
            if raw.dtype == dt:
                cq = TN.rows_norm(raw, mw.q_norm, self.cfg.norm_eps, m.q_rank, c.bufs.get("q_lat", t, mw.w_uq.k, dtype=dt), pdl=pdl)
                q_raw = N.linear(cq, mw.w_uq.w, c.bufs.get("q_up", t, mw.w_uq.n, dtype=dt), pdl=pdl)
            else:                                  # mat-vec decode: raw is fp32 beside bf16 weights
                q_raw = c.bufs.get("q_up32", t, mw.w_uq.n, dtype=torch.float32)
                P.norm_in_proj(raw[:, :mw.w_uq.k], mw.q_norm, self.cfg.norm_eps, m.q_rank, mw.w_uq.w, mw.w_uq.n, 0.0, 0.0, q_raw,
                               None, pdl=pdl)
        down = raw[:, mw.down_at:] if mw.c_norm is not None else None
        q = c.bufs.get("q", t, m.heads, mw.dim_p + mw.rot_p, dtype=dt)
        q_abs = c.bufs.get("q_abs", t, m.heads, mw.lat_p + mw.rot_p, dtype=dt)
        attn = c.bufs.get("attn", t, m.heads, mw.vdim_p, dtype=dt)
        expand = b is not None and b.latent_tiles is not None and self.latent_prefill(mw)
        some_absorbed = not expand or b.absorbed is not None
        N.latent_append(q_raw, down, mw.c_norm, self.cfg.norm_eps, mw.inv_freq, q, q_abs if some_absorbed else None, pool,
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

    # ------------------------------------------------------------------ feed-forward
    def dense_act(self, fw: DenseFfWeights, h: torch.Tensor, c: StepContext) -> torch.Tensor:
        """Gate and up projections with the gated activation."""
        t, dt, ffp = c.t, self.dtype, fw.w_down.k
        scratch = c.bufs.get("gate_up", t, 2 * ffp, dtype=dt) if dt == torch.float32 else None
        return N.gated_linear(h, fw.w_gu, fw.spec.limit, c.bufs.get("ff", t, ffp, dtype=dt), scratch, pdl=c.pdl)

    def routing(self, fw: RoutedFfWeights, c: StepContext) -> R.Routing:
        f, t = fw.spec, c.t
        i32, slots, experts = dict(dtype=torch.int32), f.top + fw.always, f.experts + fw.always
        return R.Routing(c.bufs.get("route_idx", t, slots, **i32), c.bufs.get("route_w", t, slots, dtype=torch.float32),
                         c.bufs.get("route_id", t, dtype=torch.float32) if fw.correction is not None else None,
                         c.bufs.get("route_counts", 1, experts, **i32)[0], c.bufs.get("route_offsets", 1, experts + 1, **i32)[0],
                         c.bufs.get("route_rows", t, slots, **i32))

    def router_logits(self, fw: RoutedFfWeights, h: torch.Tensor, c: StepContext) -> torch.Tensor:
        return P.logits_f32(h, fw.router, c.bufs.get("route_z", c.t, fw.router.shape[0], dtype=torch.float32))

    def expert_rows(self, fw: RoutedFfWeights, h: torch.Tensor, r: R.Routing, c: StepContext) -> torch.Tensor:
        """The chosen experts' outputs, one row per (token, slot) sorted by expert."""
        f, t, dt, pdl, ffp, slots = fw.spec, c.t, self.dtype, c.pdl, fw.w_down.k, r.idx.shape[1]
        rows = lambda name, n: c.bufs.get(name, t, slots, n, dtype=dt).view(t * slots, n)      # noqa: E731
        xs, act, y = rows("xs", self.width_p), rows("moe_act", ffp), rows("moe_y", fw.w_down.n)
        R.route_scatter(h, r, xs, fw.always, pdl=pdl)
        scratch = rows("moe_gu", 2 * ffp) if dt == torch.float32 else None
        R.grouped_gated_ffn(xs, r.offsets, fw.w_gu, fw.w_down, f.limit, t, scratch, act, y, pdl=pdl)
        return y

    def logits(self, x: torch.Tensor, h: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None,
               pdl: bool = False) -> torch.Tensor:
        """Final norm + LM head of fp32 residual rows [R, width_p] -> fp32 [R, vocab]."""
        w, r = self.w, x.shape[0]
        if out is None:
            out = torch.empty(r, self.cfg.vocab_size, dtype=torch.float32, device=self.device)
        if h is None:
            h = torch.empty(r, self.width_p, dtype=self.dtype, device=self.device)
        self.final_rows(x, h, pdl=pdl)
        return P.logits_f32(h, w.lm_head.w, out=out)

    def final_rows(self, x: torch.Tensor, h: torch.Tensor, pdl: bool = False) -> None:
        """h = the final norm of the residual rows."""
        P.rms_norm_f32(x, self.w.final_norm, self.cfg.norm_eps, h, self.cfg.width, pdl=pdl)

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
            raise _lib.NativeError(f"{self.title} runs on this package's CUDA kernels only")
        batch = RaggedBatch.plan(entries, cache, self._min_heads, self._absorb)
        for e, l in zip(batch.entries, batch.lens):
            cache.reserve(e.seq_id, l)
        batch.upload(self.device)
        bufs = self._buffers(batch.num_tokens)
        acts = self.start(batch.tokens, bufs)
        x = acts[0]
        c = StepContext(batch.num_tokens, bufs, cache, cache.block_table, batch.positions, batch.token_seq, batch.token_seq,
                        batch.runs, batch)
        for li in range(len(self.w.layers)):
            self.layer(li, acts, c)
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

    def config(self):
        return self.cfg
