"""Operations of parallel-block decoders (one norm, attention and feed-forward side by side, fp32
residual): csrc/kernels/parallel_rows.cu, parallel_gemv.cu, gemm_tcgen05.cu (split and dual
epilogues), gemm_f32.cu, and the attention kernels that take score modifiers
(flash_prefill_tc.cu, flash_decode_scored.cu, attention_any.cu).

Activations are bf16 or fp32; the dtype of the tensors picks the kernels. Row widths are padded to
multiples of eight (``pad8``)."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import _lib
from .gemm import GemmStatus, gemm_bf16_f32

_lib.register_cuda_sigs({
    "rmlx_embed_scaled": ("pppfiiiiiip", "i"),
    "rmlx_rms_norm_f32": ("pppiiifiip", "i"),
    "rmlx_qk_norm_append": ("pippfppppppiiiiiiiiiiip", "i"),
    "rmlx_parallel_gemv_max_rows": ("i", "i"),
    "rmlx_parallel_in": ("ppipfipiipiiiiffip", "i"),
    "rmlx_parallel_out": ("pppipipppiiiiiip", "i"),
    "rmlx_gemm_bf16_split_xielu": ("ppppiffiiiiiiiipip", "i"),
    "rmlx_gemm_bf16_dual_add": ("ppiiippiiipppiiiipip", "i"),
    "rmlx_sgemm": ("pipipiiiiip", "i"),
    "rmlx_sgemm_split_xielu": ("pipipiipiffiiiip", "i"),
    "rmlx_sgemm_scaled_add": ("pipippiiiiip", "i"),
    "rmlx_attention_any": ("pppppppipiiiiiiiiiii" "ffpppp" "pi" "iifff" "iip", "i"),
    "rmlx_flash_prefill_scored_supported": ("ii", "i"),
    "rmlx_flash_prefill_scored": ("ppppipipiiiiiiiiffpppp" "piipip", "i"),
    "rmlx_flash_prefill_diff": ("ppppipipiiiiiiiiiffff" "pip", "i"),
    "rmlx_flash_decode_scored_supported": ("ii", "i"),
    "rmlx_flash_decode_scored_part_o_elems": ("iiiii", "q"),
    "rmlx_flash_decode_scored_part_ml_elems": ("iiii", "q"),
    "rmlx_flash_decode_scored_ticket_elems": ("iii", "q"),
    "rmlx_flash_decode_scored": ("ppippfpppppppppp" "iiiiiiiiiii" "ffpppp" "piii" "ppif" "iifff" "ip", "i"),
})


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


@dataclass
class ScoreMods:
    """What happens to q . k before the softmax (csrc/common/score_mod.cuh); every tensor is fp32
    ``[heads]`` on the device, None switches that part off."""
    scale: float
    softcap: float = 0.0
    temp: Optional[torch.Tensor] = None
    r1: Optional[torch.Tensor] = None
    r2: Optional[torch.Tensor] = None
    sink: Optional[torch.Tensor] = None

    def args(self):
        return (self.scale, self.softcap, _lib.ptr(self.temp), _lib.ptr(self.r1), _lib.ptr(self.r2),
                _lib.ptr(self.sink))


@dataclass
class MapDiff:
    """Differential attention: a head's result is ``scale`` times the RMS norm of its first map's attention minus
    ``weight`` times its second map's."""
    weight: float
    scale: float
    eps: float

    def args(self):
        return (self.weight, self.scale, self.eps)


NO_DIFF = MapDiff(0.0, 1.0, 0.0)


def _f32(t: torch.Tensor) -> int:
    if t.dtype not in (torch.float32, torch.bfloat16):
        raise _lib.NativeError(f"these kernels take bf16 or fp32, not {t.dtype}")
    return int(t.dtype == torch.float32)


def embed_scaled(table: torch.Tensor, ids: torch.Tensor, scale: float, x: torch.Tensor, pdl: bool = False) -> torch.Tensor:
    """x[t] = table[ids[t]] * scale; table [V, D], x fp32 [T, ldx >= D] (zero from D on)."""
    _lib.require_cuda_tensor(table, ids, x)
    assert ids.dtype == torch.int32 and x.dtype == torch.float32 and table.is_contiguous() and x.is_contiguous()
    assert x.shape[0] == ids.numel()
    rc = _lib.cuda().rmlx_embed_scaled(table.data_ptr(), ids.data_ptr(), x.data_ptr(), scale, ids.numel(),
                                       table.shape[1], x.shape[1], table.shape[0], _f32(table), int(pdl),
                                       _lib.stream_ptr())
    _lib.check(rc, "embed_scaled")
    return x


def rms_norm_f32(x: torch.Tensor, w: torch.Tensor, eps: float, out: torch.Tensor, width: int, pdl: bool = False) -> torch.Tensor:
    """RMSNorm of fp32 rows; the mean is over the first ``width`` columns (the rest are zero)."""
    _lib.require_cuda_tensor(x, w, out)
    assert x.dtype == torch.float32 and w.dtype == torch.float32 and w.numel() == x.shape[1]
    assert x.is_contiguous() and out.is_contiguous() and out.shape == x.shape
    rc = _lib.cuda().rmlx_rms_norm_f32(x.data_ptr(), w.data_ptr(), out.data_ptr(), x.shape[0], width, x.shape[1],
                                       eps, _f32(out), int(pdl), _lib.stream_ptr())
    _lib.check(rc, "rms_norm_f32")
    return out


def in_proj(h: torch.Tensor, w: torch.Tensor, n_raw: int, ap: float, an: float, raw: torch.Tensor,
            act: Optional[torch.Tensor], pdl: bool = False) -> None:
    """[raw | z] = h w^T, act = xIELU(z): rows of ``w`` before ``n_raw`` give ``raw`` [T, n_raw], the
    others ``act`` [T, N - n_raw]. bf16: the tcgen05 GEMM (n_raw a multiple of 32); fp32: FFMA."""
    _lib.require_cuda_tensor(h, w, raw, act)
    t, k = h.shape
    n = w.shape[0]
    assert w.shape[1] == k and raw.shape == (t, n_raw) and (n == n_raw or act.shape == (t, n - n_raw))
    ldact = 0 if act is None else act.stride(0)
    if _f32(h):
        rc = _lib.cuda().rmlx_sgemm_split_xielu(h.data_ptr(), h.stride(0), w.data_ptr(), w.stride(0), raw.data_ptr(),
                                                raw.stride(0), n_raw, _lib.ptr(act), ldact, ap, an, t, n, k, int(pdl),
                                                _lib.stream_ptr())
    else:
        rc = _lib.cuda().rmlx_gemm_bf16_split_xielu(h.data_ptr(), w.data_ptr(), raw.data_ptr(), _lib.ptr(act), n_raw,
                                                    ap, an, t, n, k, h.stride(0), w.stride(0), raw.stride(0), ldact, 0,
                                                    GemmStatus.get(h.device).data_ptr(), int(pdl), _lib.stream_ptr())
    _lib.check(rc, "in_proj")


def out_proj_add(a: torch.Tensor, wo: torch.Tensor, ls1: torch.Tensor, act: Optional[torch.Tensor],
                 wd: Optional[torch.Tensor], ls2: Optional[torch.Tensor], x: torch.Tensor, pdl: bool = False) -> None:
    """x += ls1 * (a wo^T) + ls2 * (act wd^T) on the fp32 residual, in place."""
    _lib.require_cuda_tensor(a, wo, x, act, wd)
    t, k1 = a.shape
    n = wo.shape[0]
    assert x.dtype == torch.float32 and x.shape == (t, n) and wo.shape[1] == k1
    k2 = 0 if wd is None else wd.shape[1]
    assert k2 == 0 or (act.shape == (t, k2) and wd.shape[0] == n)
    lib, st = _lib.cuda(), _lib.stream_ptr()
    if _f32(a):
        rc = lib.rmlx_sgemm_scaled_add(a.data_ptr(), a.stride(0), wo.data_ptr(), wo.stride(0), ls1.data_ptr(),
                                       x.data_ptr(), x.stride(0), t, n, k1, int(pdl), st)
        _lib.check(rc, "out_proj_add")
        if k2:
            rc = lib.rmlx_sgemm_scaled_add(act.data_ptr(), act.stride(0), wd.data_ptr(), wd.stride(0), ls2.data_ptr(),
                                           x.data_ptr(), x.stride(0), t, n, k2, int(pdl), st)
            _lib.check(rc, "out_proj_add")
        return
    rc = lib.rmlx_gemm_bf16_dual_add(a.data_ptr(), wo.data_ptr(), k1, a.stride(0), wo.stride(0),
                                     _lib.ptr(act) if k2 else None, _lib.ptr(wd), k2, act.stride(0) if k2 else 0,
                                     wd.stride(0) if k2 else 0, ls1.data_ptr(), _lib.ptr(ls2), x.data_ptr(),
                                     x.stride(0), t, n, 0, GemmStatus.get(a.device).data_ptr(), int(pdl), st)
    _lib.check(rc, "out_proj_add")


def logits_f32(h: torch.Tensor, w: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """h w^T as fp32 (bf16 operands: the tensor-core accumulator unrounded)."""
    if not _f32(h):
        return gemm_bf16_f32(h, w, out=out)
    _lib.require_cuda_tensor(h, w)
    t, k = h.shape
    if out is None:
        out = torch.empty(t, w.shape[0], dtype=torch.float32, device=h.device)
    rc = _lib.cuda().rmlx_sgemm(h.data_ptr(), h.stride(0), w.data_ptr(), w.stride(0), out.data_ptr(), out.stride(0),
                                t, w.shape[0], k, 0, _lib.stream_ptr())
    _lib.check(rc, "sgemm")
    return out


def gemv_max_rows(k: int) -> int:
    """Rows one launch of the decode projections takes for staged widths adding up to ``k``."""
    return int(_lib.cuda().rmlx_parallel_gemv_max_rows(k))


def norm_in_proj(x: torch.Tensor, norm_w: torch.Tensor, eps: float, width: int, w: torch.Tensor, n_raw: int,
                 ap: float, an: float, raw: torch.Tensor, act: Optional[torch.Tensor], pdl: bool = False) -> None:
    """Decode form of ``rms_norm_f32`` + ``in_proj``: fp32 residual rows in, raw rows out in fp32."""
    _lib.require_cuda_tensor(x, norm_w, w, raw, act)
    b, k = x.shape
    n = w.shape[0]
    assert x.dtype == torch.float32 and raw.dtype == torch.float32 and w.dtype == torch.bfloat16
    assert w.is_contiguous() and w.shape[1] == k and norm_w.numel() == k
    step = gemv_max_rows(k)
    for b0 in range(0, b, max(step, 1)):
        bb = min(step, b - b0)
        rc = _lib.cuda().rmlx_parallel_in(
            w.data_ptr(), x[b0:].data_ptr(), x.stride(0), norm_w.data_ptr(), eps, width, raw[b0:].data_ptr(),
            raw.stride(0), n_raw, None if act is None else act[b0:].data_ptr(), 0 if act is None else act.stride(0),
            bb, n, k, ap, an, int(pdl), _lib.stream_ptr())
        _lib.check(rc, "parallel_in")


def gemv_out_add(a: torch.Tensor, wo: torch.Tensor, ls1: torch.Tensor, act: Optional[torch.Tensor],
                 wd: Optional[torch.Tensor], ls2: Optional[torch.Tensor], x: torch.Tensor, pdl: bool = False) -> None:
    """Decode form of ``out_proj_add``."""
    _lib.require_cuda_tensor(a, wo, x, act, wd)
    b, k1 = a.shape
    k2 = 0 if wd is None else wd.shape[1]
    assert a.dtype == torch.bfloat16 and wo.is_contiguous() and (wd is None or wd.is_contiguous())
    step = gemv_max_rows(k1 + k2)
    for b0 in range(0, b, max(step, 1)):
        bb = min(step, b - b0)
        rc = _lib.cuda().rmlx_parallel_out(
            wo.data_ptr(), _lib.ptr(wd), a[b0:].data_ptr(), a.stride(0), act[b0:].data_ptr() if k2 else None,
            act.stride(0) if k2 else 0, ls1.data_ptr(), _lib.ptr(ls2), x[b0:].data_ptr(), x.stride(0), bb,
            wo.shape[0], k1, k2, int(pdl), _lib.stream_ptr())
        _lib.check(rc, "parallel_out")


def qk_norm_append(raw: torch.Tensor, q_w: torch.Tensor, k_w: torch.Tensor, eps: float, q: torch.Tensor,
                   k_cache: torch.Tensor, v_cache: torch.Tensor, block_table: torch.Tensor, positions: torch.Tensor,
                   token_seq: Optional[torch.Tensor], heads: int, dim: int, vdim: int, pdl: bool = False) -> None:
    """Whole-projection RMS norm of queries and keys; q [T, H, pad8(dim)], keys / values to their pages."""
    _lib.require_cuda_tensor(raw, q, k_cache, v_cache, block_table, positions, token_seq)
    t = raw.shape[0]
    hkv, page = k_cache.shape[1], k_cache.shape[2]
    assert q.shape == (t, heads, k_cache.shape[3]) and q.dtype == raw.dtype == k_cache.dtype == v_cache.dtype
    assert q_w.numel() == heads * dim and k_w.numel() == hkv * dim and q_w.dtype == torch.float32
    assert block_table.dtype == positions.dtype == torch.int32
    rc = _lib.cuda().rmlx_qk_norm_append(
        raw.data_ptr(), raw.stride(0), q_w.data_ptr(), k_w.data_ptr(), eps, q.data_ptr(), k_cache.data_ptr(),
        v_cache.data_ptr(), block_table.data_ptr(), positions.data_ptr(), _lib.ptr(token_seq), t, heads, hkv, dim,
        vdim, k_cache.shape[3], v_cache.shape[3], block_table.stride(0), page, _f32(raw), int(pdl), _lib.stream_ptr())
    _lib.check(rc, "qk_norm_append")


def _gate_args(gate: Optional[torch.Tensor], t: int, h: int, dtype):
    if gate is None:
        return None, 0
    assert gate.shape == (t, h) and gate.stride(1) == 1 and gate.dtype == dtype
    return gate.data_ptr(), gate.stride(0)


def prefill_scored_supported(dk: int, dv: int) -> bool:
    return bool(_lib.cuda().rmlx_flash_prefill_scored_supported(dk, dv))


def decode_scored_supported(dk: int, dv: int) -> bool:
    return bool(_lib.cuda().rmlx_flash_decode_scored_supported(dk, dv))


def flash_prefill_scored(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, block_table: torch.Tensor,
                         tiles: torch.Tensor, mods: ScoreMods, out: torch.Tensor, window: int = 0, lanes: int = 1,
                         gate: Optional[torch.Tensor] = None, chunk: int = 0, pdl: bool = False) -> torch.Tensor:
    """Ragged causal attention over pages on the tensor cores: q [T, H, dk] bf16; ``tiles`` int32
    [n, 4] = (first row, rows <= lanes * 128, position of the first row, row of ``block_table``).
    ``gate`` [T, H]: logits of a sigmoid each head's output is multiplied by. ``chunk`` > 0: a query sees only the
    keys of its own chunk of so many positions, counted from the sequence's start."""
    _lib.require_cuda_tensor(q, k_cache, v_cache, block_table, tiles, out)
    t, h, dk = q.shape
    assert q.is_contiguous() and out.is_contiguous() and tiles.dtype == torch.int32 and tiles.is_contiguous()
    assert k_cache.shape[2] == 16 and k_cache.shape[3] == dk and out.shape == (t, h, v_cache.shape[3])
    rc = _lib.cuda().rmlx_flash_prefill_scored(
        q.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), block_table.data_ptr(), block_table.stride(0),
        tiles.data_ptr(), tiles.shape[0], out.data_ptr(), t, h, k_cache.shape[1], dk, v_cache.shape[3],
        k_cache.shape[0], window, chunk, *mods.args(), *_gate_args(gate, t, h, q.dtype), lanes, GemmStatus.get(q.device).data_ptr(), int(pdl),
        _lib.stream_ptr())
    _lib.check(rc, "flash_prefill_scored")
    return out


def flash_prefill_diff(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, block_table: torch.Tensor,
                       tiles: torch.Tensor, scale: float, diff: MapDiff, vdim: int, out: torch.Tensor, window: int = 0,
                       chunk: int = 0, pdl: bool = False) -> torch.Tensor:
    """``flash_prefill_scored`` for differential attention: q [T, H, 2, dk], key rows of two keys, out [T, H, dv]; tiles of
    at most 128 rows."""
    _lib.require_cuda_tensor(q, k_cache, v_cache, block_table, tiles, out)
    t, h, maps, dk = q.shape
    assert maps == 2 and q.is_contiguous() and out.is_contiguous() and tiles.dtype == torch.int32 and tiles.is_contiguous()
    assert k_cache.shape[2] == 16 and k_cache.shape[3] == 2 * dk and out.shape == (t, h, v_cache.shape[3])
    rc = _lib.cuda().rmlx_flash_prefill_diff(
        q.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), block_table.data_ptr(), block_table.stride(0),
        tiles.data_ptr(), tiles.shape[0], out.data_ptr(), t, h, k_cache.shape[1], dk, v_cache.shape[3], vdim,
        k_cache.shape[0], window, chunk, scale, *diff.args(), GemmStatus.get(q.device).data_ptr(), int(pdl), _lib.stream_ptr())
    _lib.check(rc, "flash_prefill_diff")
    return out


class ScoredDecodeScratch:
    """Split-KV scratch of ``flash_decode_scored`` for up to ``rows`` rows (differential attention: twice the heads)."""

    def __init__(self, rows: int, heads: int, kv_heads: int, dv: int, splits: int, device):
        lib = _lib.cuda()
        self.splits = splits
        self.part_o = torch.empty(lib.rmlx_flash_decode_scored_part_o_elems(rows, heads, kv_heads, splits, dv),
                                  dtype=torch.float32, device=device)
        self.part_ml = torch.empty(lib.rmlx_flash_decode_scored_part_ml_elems(rows, heads, kv_heads, splits),
                                   dtype=torch.float32, device=device)
        self.tickets = torch.zeros(lib.rmlx_flash_decode_scored_ticket_elems(rows, heads, kv_heads),
                                   dtype=torch.int32, device=device)


def flash_decode_scored(k_cache: torch.Tensor, v_cache: torch.Tensor, block_table: torch.Tensor,
                        positions: torch.Tensor, mods: ScoreMods, out: torch.Tensor, scratch: ScoredDecodeScratch,
                        heads: int, dim: int, vdim: int, q: Optional[torch.Tensor] = None,
                        raw: Optional[torch.Tensor] = None, q_w: Optional[torch.Tensor] = None,
                        k_w: Optional[torch.Tensor] = None, eps: float = 0.0, rows: Optional[torch.Tensor] = None,
                        table_rows: Optional[torch.Tensor] = None, n_rows: Optional[int] = None, window: int = 0,
                        gate: Optional[torch.Tensor] = None, head_norm: bool = False, gate_col: int = -1,
                        chunk: int = 0, bias: Optional[torch.Tensor] = None, inv_freq: Optional[torch.Tensor] = None,
                        grow: float = 1.0, neighbours: bool = False, normed: bool = True, diff: Optional[MapDiff] = None,
                        pdl: bool = False) -> torch.Tensor:
    """One token per row: q [T, H, dk] (keys already appended) or the fused form on the un-normalised
    fp32 projection ``raw`` [T, >= q|k|v], which also appends the key and value (``head_norm``: the
    norms are per head, their weights [dim] or None; with it ``bias`` is added to the projection, and the first
    ``2 * inv_freq.numel()`` values of query and key heads rotate, i with i + pairs or (``neighbours``) 2 i with 2 i + 1,
    before the norm, which ``normed`` False leaves out; ``gate_col``: where the output gate's logits start in a row).
    ``rows`` int32: the batch rows to run (default: the first ``n_rows``). ``diff``: differential attention, q [T, H, 2, dk]
    or raw rows [q: H x 2 x dim | k: Hkv x 2 x dim | v] with ``head_norm``, key rows of two keys."""
    _lib.require_cuda_tensor(k_cache, v_cache, block_table, positions, out, q, raw)
    src = q if q is not None else raw
    n = rows.numel() if rows is not None else (n_rows or src.shape[0])
    maps = 1 if diff is None else 2
    dk = k_cache.shape[3] // maps
    assert k_cache.shape[2] == 16 and out.is_contiguous() and k_cache.dtype == torch.bfloat16
    assert q is None or (q.is_contiguous() and q.shape[1:] == ((heads, dk) if maps == 1 else (heads, 2, dk)))
    assert raw is None or raw.dtype == torch.float32
    rc = _lib.cuda().rmlx_flash_decode_scored(
        _lib.ptr(q), _lib.ptr(raw), 0 if raw is None else raw.stride(0), _lib.ptr(q_w), _lib.ptr(k_w), eps,
        k_cache.data_ptr(), v_cache.data_ptr(), block_table.data_ptr(), positions.data_ptr(), _lib.ptr(rows),
        _lib.ptr(table_rows), out.data_ptr(), scratch.part_o.data_ptr(), scratch.part_ml.data_ptr(),
        scratch.tickets.data_ptr(), n, heads, k_cache.shape[1], dim, vdim, dk, v_cache.shape[3],
        block_table.stride(0), scratch.splits, window, chunk, *mods.args(),
        *_gate_args(gate, 0 if q is None else q.shape[0], heads, torch.bfloat16), (1 if normed else 2) if head_norm else 0,
        gate_col, _lib.ptr(bias), _lib.ptr(inv_freq), 0 if inv_freq is None else 2 * inv_freq.numel(), grow, int(neighbours), maps,
        *(diff or NO_DIFF).args(), int(pdl), _lib.stream_ptr())
    _lib.check(rc, "flash_decode_scored")
    return out


def attention_any(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, block_table: torch.Tensor,
                  positions: torch.Tensor, token_seq: Optional[torch.Tensor], mods: ScoreMods, out: torch.Tensor,
                  window: int = 0, gate: Optional[torch.Tensor] = None, rows: Optional[torch.Tensor] = None,
                  chunk: int = 0, diff: Optional[MapDiff] = None, vdim: int = 0, pdl: bool = False) -> torch.Tensor:
    """Attention of single query tokens over pages for any head widths, bf16 or fp32 storage. Cache rows
    may be wider than the query (key) and the output (value): ``k_cache`` and ``v_cache`` may be one
    pool whose rows hold both (latent attention). ``rows``: batch rows to run (default: all). ``diff``: differential
    attention, q [T, H, 2, dk], key rows of two keys, heads of ``vdim`` values."""
    _lib.require_cuda_tensor(q, k_cache, v_cache, block_table, positions, token_seq, out)
    t, h, dk = q.shape[0], q.shape[1], q.shape[-1]
    maps = 1 if diff is None else 2
    assert q.dim() == 2 + maps and q.is_contiguous() and out.is_contiguous() and q.dtype == k_cache.dtype == out.dtype
    assert k_cache.shape[3] >= maps * dk and out.shape[:2] == (t, h) and v_cache.shape[3] >= out.shape[2]
    rc = _lib.cuda().rmlx_attention_any(
        q.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), block_table.data_ptr(), positions.data_ptr(),
        _lib.ptr(token_seq), _lib.ptr(rows), 0 if rows is None else rows.numel(), out.data_ptr(), t, h,
        k_cache.shape[1], dk, out.shape[2], k_cache.shape[3], v_cache.shape[3], block_table.stride(0),
        k_cache.shape[2], window, chunk, *mods.args(), *_gate_args(gate, t, h, q.dtype), maps, vdim,
        *(diff or NO_DIFF).args(), _f32(q), int(pdl), _lib.stream_ptr())
    _lib.check(rc, "attention_any")
    return out
