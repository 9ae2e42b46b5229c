"""Posudra: a decoder of parallel blocks (attention and feed-forward read one norm's output and are
added to an fp32 residual stream, each with a learned layer scale) without rotary embedding.
Positions enter attention as a logarithmic distance bias; scores also have a per-head temperature, a
soft cap and a sink; queries and keys are RMS-normalised over their whole projection; the dense
feed-forward uses xIELU.

Per layer the weights are kept as three matrices: ``w_in`` = [q; k; v; up] (one projection of the
norm's output), ``w_o`` and ``w_down`` (one kernel adds both to the residual). Widths that are not
multiples of eight are zero-padded when the weights are built, so every kernel sees aligned rows.

Prompts and mixed batches run through ``forward_batch`` (a ragged batch, five launches per layer),
decode steps through ``ParallelBlockDecode`` (three launches per layer, one CUDA graph per step).
Everything runs on this package's CUDA kernels, in bf16 or (``dtype=torch.float32``) in true 32-bit;
there is no CPU path."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Dict, List, Optional, Sequence

import torch

from .. import _lib
from ..config import ParallelLayerSpec, PosudraConfig, ScoredAttentionSpec
from ..kv.paged import PAGE, PagedKvCache
from ..ops import parallel_block as P
from ..ops.decode import default_splits
from ..ops.gemm import GemmStatus
from ..ops.parallel_block import ScoreMods, pad8
from ..ops.weights import LinearWeight, W_BF16
from .ragged import Entry, RaggedBatch
from .weights import ParallelLayout


def posudra_tiny() -> PosudraConfig:
    """Test-size preset; the layers differ in every size, one has no feed-forward."""
    return PosudraConfig(vocab_size=301, width=96, norm_eps=1e-5, embedding_scale=3.0, layers=[
        ParallelLayerSpec(ScoredAttentionSpec(6, 2, 32, 40, 0.2, 20.0), 160),
        ParallelLayerSpec(ScoredAttentionSpec(2, 2, 72, 16, 0.15, 30.0), 0),
        ParallelLayerSpec(ScoredAttentionSpec(4, 1, 24, 64, 0.25, 15.0), 200)]).validate()


def posudra_8b(num_layers: int = 32) -> PosudraConfig:
    """Layers of the size of an 8B dense decoder (benchmarks)."""
    layer = ParallelLayerSpec(ScoredAttentionSpec(32, 8, 128, 128, 128 ** -0.5, 50.0), 21504)
    return PosudraConfig(vocab_size=128256, width=4096, layers=[layer] * num_layers, norm_eps=1e-6,
                         embedding_scale=1.0, name="posudra-8b").validate()


# ------------------------------------------------------------------------------------------------
# Weights
# ------------------------------------------------------------------------------------------------
@dataclass
class ParallelLayerWeights:
    spec: ParallelLayerSpec
    norm1: torch.Tensor              # fp32 [width_p]
    w_in: LinearWeight               # [n_raw + ff_p, width_p]: q | k | v (zero rows up to n_raw) | up
    n_raw: int                       # multiple of 32
    w_o: LinearWeight                # [width_p, heads * pad8(vdim)]
    w_down: Optional[LinearWeight]   # [width_p, ff_p]
    q_norm: torch.Tensor             # fp32 [heads * dim]
    k_norm: torch.Tensor             # fp32 [kv_heads * dim]
    mods: ScoreMods
    ls1: torch.Tensor                # fp32 [width_p]
    ls2: Optional[torch.Tensor]
    act_p: float = 0.0               # xIELU's quadratic factors, softplus already applied
    act_n: float = 0.0

    @property
    def ff(self) -> int:
        return 0 if self.w_down is None else self.w_down.k


@dataclass
class PosudraWeights:
    cfg: PosudraConfig
    embed: torch.Tensor              # [vocab, width]
    layers: List[ParallelLayerWeights]
    final_norm: torch.Tensor         # fp32 [width_p]
    lm_head: LinearWeight            # [vocab, width_p]
    layout: ParallelLayout
    vocab_base: int = 0

    def nbytes(self) -> int:
        t = self.embed.numel() * self.embed.element_size() + self.lm_head.nbytes()
        return t + sum(w.nbytes() for l in self.layers for w in (l.w_in, l.w_o, l.w_down) if w is not None)


def tensor_shapes(cfg: PosudraConfig) -> Dict[str, tuple]:
    """Checkpoint tensor names and shapes."""
    d = cfg.width
    out = {"embed": (cfg.vocab_size, d)}
    for i, l in enumerate(cfg.layers):
        m, p = l.mixer, f"l{i}."
        out.update({p + "norm1": (d,), p + "mix.q": (m.heads * m.dim, d), p + "mix.k": (m.kv_heads * m.dim, d),
                    p + "mix.v": (m.kv_heads * m.vdim, d), p + "mix.q.norm": (m.heads * m.dim,),
                    p + "mix.k.norm": (m.kv_heads * m.dim,), p + "mix.r1": (m.heads,), p + "mix.r2": (m.heads,),
                    p + "mix.temp": (m.heads,), p + "mix.sink": (m.heads,), p + "mix.o": (d, m.heads * m.vdim),
                    p + "ls1": (d,)})
        if l.ff:
            out.update({p + "mlp.up": (l.ff, d), p + "mlp.down": (d, l.ff), p + "mlp.act": (2,), p + "ls2": (d,)})
    out.update({"final.norm": (d,), "head": (cfg.vocab_size, d)})
    return out


def random_tensors(cfg: PosudraConfig, seed: int = 0, device="cpu", dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Random checkpoint tensors of the design (projections scaled by 1 / sqrt(inputs))."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".", 1)[-1]
        x = torch.randn(*shape, generator=g, device=device, dtype=torch.float32 if len(shape) == 1 else dtype)
        if leaf in ("norm1", "mix.q.norm", "mix.k.norm", "norm"):
            x = 1.0 + 0.2 * x
        elif leaf in ("ls1", "ls2"):
            x = 0.5 + 0.1 * x
        elif leaf == "mix.r1":
            x = 0.2 + 0.5 * x.abs()
        elif leaf == "mix.r2":
            x = 0.1 + 0.2 * x.abs()
        elif leaf == "mix.temp":
            x = 1.0 + 0.2 * x
        elif len(shape) == 2 and name != "embed":
            x = x * shape[1] ** -0.5
        out[name] = x.to(dtype)
    return out


def build_weights(cfg: PosudraConfig, tensors: Dict[str, torch.Tensor], device="cpu", dtype=torch.bfloat16
                  ) -> PosudraWeights:
    """Runtime weights from checkpoint tensors: projections merged and padded, per-channel vectors in
    fp32, everything on ``device``."""
    if dtype not in (torch.bfloat16, torch.float32):
        raise ValueError("Posudra runs in bfloat16 or float32")
    want = tensor_shapes(cfg)
    for name, shape in want.items():
        if name not in tensors:
            raise KeyError(f"checkpoint has no tensor {name!r}")
        if tuple(tensors[name].shape) != shape:
            raise ValueError(f"{name}: shape {tuple(tensors[name].shape)}, expected {shape}")
    wp = pad8(cfg.width)

    def mat(parts, rows: int, cols: int) -> LinearWeight:
        """Stack ``parts`` ((row offset, tensor) pairs) into a zero [rows, cols] matrix."""
        out = torch.zeros(rows, cols, dtype=dtype, device=device)
        for at, t in parts:
            out[at:at + t.shape[0], :t.shape[1]] = t.to(device=device, dtype=dtype)
        return LinearWeight(W_BF16, out)

    def vec(t, n: Optional[int] = None) -> torch.Tensor:
        out = torch.zeros(n or t.numel(), dtype=torch.float32, device=device)
        out[:t.numel()] = t.to(device=device, dtype=torch.float32)
        return out

    layers = []
    for i, spec in enumerate(cfg.layers):
        m, p = spec.mixer, f"l{i}."
        g = lambda n: tensors[p + n]                                     # noqa: B023,E731
        nq, nk, nv = m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim
        n_raw, ffp, dvp = (nq + nk + nv + 31) // 32 * 32, pad8(spec.ff), pad8(m.vdim)
        parts = [(0, g("mix.q")), (nq, g("mix.k")), (nq + nk, g("mix.v"))]
        if spec.ff:
            parts.append((n_raw, g("mlp.up")))
        # attention writes heads at stride pad8(vdim): spread the output projection's columns likewise
        wo = torch.zeros(cfg.width, m.heads, dvp, dtype=dtype, device=device)
        wo[:, :, :m.vdim] = g("mix.o").to(device=device, dtype=dtype).view(cfg.width, m.heads, m.vdim)
        ap = an = 0.0
        if spec.ff:
            a = torch.nn.functional.softplus(g("mlp.act").detach().to("cpu", torch.float32))
            ap, an = float(a[0]), 0.5 + float(a[1])
        layers.append(ParallelLayerWeights(
            spec=spec, norm1=vec(g("norm1"), wp), w_in=mat(parts, n_raw + ffp, wp), n_raw=n_raw,
            w_o=mat([(0, wo.view(cfg.width, -1))], wp, m.heads * dvp),
            w_down=mat([(0, g("mlp.down"))], wp, ffp) if spec.ff else None,
            q_norm=vec(g("mix.q.norm")), k_norm=vec(g("mix.k.norm")),
            mods=ScoreMods(m.scale, m.softcap, vec(g("mix.temp")), vec(g("mix.r1")), vec(g("mix.r2")),
                           vec(g("mix.sink"))),
            ls1=vec(g("ls1"), wp), ls2=vec(g("ls2"), wp) if spec.ff else None, act_p=ap, act_n=an))
    return PosudraWeights(cfg=cfg, embed=tensors["embed"].to(device=device, dtype=dtype).contiguous(), layers=layers,
                          final_norm=vec(tensors["final.norm"], wp), lm_head=mat([(0, tensors["head"])], cfg.vocab_size, wp),
                          layout=ParallelLayout())


def save_checkpoint(model_dir: str, cfg: PosudraConfig, tensors: Dict[str, torch.Tensor]) -> None:
    """config.json and model.safetensors of a Posudra model."""
    from safetensors.torch import save_file
    os.makedirs(model_dir, exist_ok=True)
    save_file({k: v.to(torch.bfloat16).contiguous().cpu() for k, v in tensors.items()},
              os.path.join(model_dir, "model.safetensors"))
    with open(os.path.join(model_dir, "config.json"), "w") as f:
        json.dump(cfg.to_json(), f, indent=1)


# ------------------------------------------------------------------------------------------------
# Model
# ------------------------------------------------------------------------------------------------
class BlockBuffers:
    """Activations of up to ``rows`` tokens, allocated once and viewed per layer (layers may differ)."""

    def __init__(self, model: "PosudraModel", rows: int, raw_f32: bool = False):
        w, dt, dev = model.w, model.dtype, model.device
        wp = model.width_p
        self.rows = rows
        self.x = torch.empty(rows, wp, dtype=torch.float32, device=dev)
        self.h = torch.empty(rows, wp, dtype=dt, device=dev)

        def flat(per_row: int, dtype) -> torch.Tensor:
            return torch.empty(rows * max(per_row, 8), dtype=dtype, device=dev)

        specs = [l.spec.mixer for l in w.layers]
        self._raw = flat(max(l.n_raw for l in w.layers), dt)
        self._raw32 = flat(max(l.n_raw for l in w.layers), torch.float32) if raw_f32 else None
        self._act = flat(max(l.ff for l in w.layers), dt)
        self._q = flat(max(m.heads * pad8(m.dim) for m in specs), dt)
        self._attn = flat(max(m.heads * pad8(m.vdim) for m in specs), dt)

    def layer(self, lw: ParallelLayerWeights, t: int):
        """(raw, act or None, q, attn) for ``t`` rows of this layer."""
        m = lw.spec.mixer
        dkp, dvp = pad8(m.dim), pad8(m.vdim)
        v = lambda buf, *s: buf[:torch.Size(s).numel()].view(*s)          # noqa: E731
        return (v(self._raw, t, lw.n_raw), v(self._act, t, lw.ff) if lw.ff else None,
                v(self._q, t, m.heads, dkp), v(self._attn, t, m.heads, dvp))

    def raw32(self, lw: ParallelLayerWeights, t: int) -> torch.Tensor:
        return self._raw32[:t * lw.n_raw].view(t, lw.n_raw)


class PosudraModel:
    """One GPU's weights and the forward passes over them."""

    # a step may hold prompt portions and decoded tokens together (``forward_batch``)
    mixed_batches = True

    def __init__(self, weights: PosudraWeights):
        self.w, self.cfg, self.layout = weights, weights.cfg, weights.layout
        self.device = weights.embed.device
        self.dtype = weights.embed.dtype
        self.width_p = pad8(self.cfg.width)
        self.allgather_logits = None
        self._bufs: Optional[BlockBuffers] = None
        self._scratch: Dict[tuple, P.ScoredDecodeScratch] = {}

    @classmethod
    def from_config(cls, cfg: Optional[PosudraConfig] = None, seed: int = 0, device="cuda", dtype=torch.bfloat16
                    ) -> "PosudraModel":
        """Random-initialised model (default: the test-size preset)."""
        cfg = cfg or posudra_tiny()
        gen_dev = device if torch.device(device).type == "cuda" and cfg.width >= 1024 else "cpu"
        return cls(build_weights(cfg, random_tensors(cfg, seed, gen_dev), device, dtype))

    @classmethod
    def from_checkpoint(cls, model_dir: str, device="cuda", dtype=torch.bfloat16) -> "PosudraModel":
        from ..loader.safetensors_loader import load_model
        weights, _cfg = load_model(model_dir, device=device, dtype=dtype)
        return cls(weights)

    # ------------------------------------------------------------------ cache
    def kv_shapes(self) -> List[tuple]:
        return [(l.mixer.kv_heads, pad8(l.mixer.dim), pad8(l.mixer.vdim)) for l in self.cfg.layers]

    def new_cache(self, num_blocks: int, max_seqs: int = 64, max_blocks_per_seq: Optional[int] = None,
                  dtype=None, kv_quant: Optional[str] = None) -> PagedKvCache:
        """``num_blocks`` pages of 16 tokens (page 0 is reserved). Without ``max_blocks_per_seq`` one
        sequence may take the whole pool, or ``cfg.max_seq_len`` tokens if that is set."""
        if kv_quant is not None:
            raise ValueError("Posudra's attention kernels read 16- or 32-bit caches")
        if max_blocks_per_seq is None:
            max_blocks_per_seq = max(1, num_blocks - 1)
            if self.cfg.max_seq_len:
                max_blocks_per_seq = min(max_blocks_per_seq, (self.cfg.max_seq_len + PAGE - 1) // PAGE)
        shapes = self.kv_shapes()
        return PagedKvCache(num_blocks, len(shapes), shapes[0][0], shapes[0][1], dtype=dtype or self.dtype,
                            device=self.device, max_seqs=max_seqs, max_blocks_per_seq=max_blocks_per_seq,
                            layer_shapes=shapes)

    def make_decode_engine(self, cache: PagedKvCache, max_batch: int, comm=None):
        from .parallel_decode import ParallelBlockDecode
        if comm is not None:
            raise ValueError("Posudra runs on one GPU")
        return ParallelBlockDecode(self, cache, max_batch=max_batch)

    # ------------------------------------------------------------------ layers
    def scratch(self, lw: ParallelLayerWeights, rows: int, splits: int) -> P.ScoredDecodeScratch:
        """Split-KV scratch, shared by every layer of the same head shape."""
        m = lw.spec.mixer
        key = (m.heads, m.kv_heads, pad8(m.vdim), rows, splits)
        if key not in self._scratch:
            self._scratch[key] = P.ScoredDecodeScratch(rows, m.heads, m.kv_heads, pad8(m.vdim), splits, self.device)
        return self._scratch[key]

    def decode_splits(self, lw: ParallelLayerWeights, rows: int, max_len: int) -> int:
        m = lw.spec.mixer
        return default_splits(rows, m.kv_heads, (m.heads // m.kv_heads + 15) // 16, max_len)

    def tensor_core_decode(self, lw: ParallelLayerWeights) -> bool:
        m = lw.spec.mixer
        return self.dtype == torch.bfloat16 and P.decode_scored_supported(pad8(m.dim), pad8(m.vdim))

    def block(self, li: int, bufs: BlockBuffers, t: int, cache: PagedKvCache, block_table, positions, token_seq,
              attend, pdl: bool = False) -> None:
        """One parallel block over ``t`` rows of ``bufs.x``: norm, merged projection (+ xIELU), query /
        key norm + append, ``attend(lw, q, attn)``, both output projections into the residual."""
        lw, eps, m = self.w.layers[li], self.cfg.norm_eps, self.w.layers[li].spec.mixer
        raw, act, q, attn = bufs.layer(lw, t)
        x, h = bufs.x[:t], bufs.h[:t]
        P.rms_norm_f32(x, lw.norm1, eps, h, self.cfg.width, pdl=pdl)
        P.in_proj(h, lw.w_in.w, lw.n_raw, lw.act_p, lw.act_n, raw, act, pdl=pdl)
        P.qk_norm_append(raw, lw.q_norm, lw.k_norm, eps, q, cache.k[li], cache.v[li], block_table, positions,
                         token_seq, m.heads, m.dim, m.vdim, pdl=pdl)
        attend(lw, q, attn)
        P.out_proj_add(attn.view(t, -1), lw.w_o.w, lw.ls1, act, None if lw.w_down is None else lw.w_down.w, lw.ls2,
                       x, pdl=pdl)

    def logits(self, x: torch.Tensor, h: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None,
               pdl: bool = False) -> torch.Tensor:
        """Final norm + LM head of fp32 residual rows [R, width_p] -> fp32 [R, vocab]."""
        w, r, v = self.w, x.shape[0], self.cfg.vocab_size
        if out is None:
            out = torch.empty(r, v, dtype=torch.float32, device=self.device)
        if self.dtype == torch.bfloat16 and r <= 4 and P.gemv_max_rows(self.width_p) > 0:
            P.norm_in_proj(x, w.final_norm, self.cfg.norm_eps, self.cfg.width, w.lm_head.w, v, 0.0, 0.0, out, None, pdl=pdl)
            return out
        if h is None:
            h = torch.empty(r, self.width_p, dtype=self.dtype, device=self.device)
        P.rms_norm_f32(x, w.final_norm, self.cfg.norm_eps, h, self.cfg.width, pdl=pdl)
        return P.logits_f32(h, w.lm_head.w, out=out)

    # ------------------------------------------------------------------ ragged batches
    def _buffers(self, rows: int) -> BlockBuffers:
        if self._bufs is None or self._bufs.rows < rows:
            self._bufs = None
            self._bufs = BlockBuffers(self, max(rows, 256))
        return self._bufs

    @torch.no_grad()
    def forward_batch(self, entries: Sequence[Entry], cache: PagedKvCache, observe=None) -> torch.Tensor:
        """Run the entries' tokens as one batch on top of what the cache holds; returns the wanted
        logits, fp32 [wanted, vocab], in the order of the entries and their ``want``. ``observe``:
        called with (layer, residual rows [T, width]) after every layer."""
        if self.device.type != "cuda":
            raise _lib.NativeError("Posudra runs on this package's CUDA kernels only")
        batch = RaggedBatch.plan(entries, cache, min(l.mixer.heads for l in self.cfg.layers))
        for e, l in zip(batch.entries, batch.lens):
            cache.reserve(e.seq_id, l)
        batch.upload(self.device)
        t = batch.num_tokens
        bufs = self._buffers(t)
        x = bufs.x[:t]
        P.embed_scaled(self.w.embed, batch.tokens, self.cfg.embedding_scale, x)

        for li in range(len(self.w.layers)):
            self.block(li, bufs, t, cache, cache.block_table, batch.positions, batch.token_seq,
                       lambda lw, q, attn: self._attend(li, lw, q, attn, batch, cache))       # noqa: B023
            if observe is not None:
                observe(li, x[:, :self.cfg.width])
        for e, l in zip(batch.entries, batch.lens):
            cache.commit(e.seq_id, l)
        if not batch.want_host:
            return torch.empty(0, self.cfg.vocab_size, dtype=torch.float32, device=self.device)
        return self.logits(x.index_select(0, batch.want.long()))

    def _attend(self, li: int, lw: ParallelLayerWeights, q, attn, batch: RaggedBatch, cache: PagedKvCache) -> None:
        m, k, v = lw.spec.mixer, cache.k[li], cache.v[li]
        dkp, dvp = k.shape[3], v.shape[3]
        if not (self.tensor_core_decode(lw) and P.prefill_scored_supported(dkp, dvp)):
            P.attention_any(q, k, v, cache.block_table, batch.positions, batch.token_seq, lw.mods, attn)
            return
        if batch.tiles is not None:
            P.flash_prefill_scored(q, k, v, cache.block_table, batch.tiles, lw.mods, attn, lanes=batch.lanes)
        if batch.single is not None:
            n = len(batch.single_host)
            splits = self.decode_splits(lw, n, batch.single_len)
            P.flash_decode_scored(k, v, cache.block_table, batch.positions, lw.mods, attn,
                                  self.scratch(lw, n, splits), m.heads, m.dim, m.vdim, q=q, rows=batch.single,
                                  table_rows=batch.token_seq)

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

    def config(self) -> PosudraConfig:
        return self.cfg
