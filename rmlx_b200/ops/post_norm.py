"""Row operations of decoders whose norms sit on the sublayers' outputs (csrc/kernels/postnorm_rows.cu),
plain projections in the activations' type, and the per-head products of absorbed latent attention
(head_gemv.cu). Activations are bf16 or fp32; the dtype of the tensors picks the kernels."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import _lib
from .gemm import gemm_bf16
from .parallel_block import _f32
from .quantized import xgemm
from .weights import LinearWeight

_lib.register_cuda_sigs({
    "rmlx_embed_norm": ("pppfppiiiiiip", "i"),
    "rmlx_post_norm_add": ("piipfppiiiiip", "i"),
    "rmlx_head_norm_append": ("piippfpppppp" "iiiiiiiiiiip", "i"),
    "rmlx_latent_append": ("pipiipfpi" "pppippp" "iiiiiiiiiiiip", "i"),
    "rmlx_gated_act": ("ppiifiip", "i"),
    "rmlx_tanh_rows": ("ppqiip", "i"),
    "rmlx_head_gemv": ("ppiipiipiiiiiip", "i"),
    "rmlx_postnorm_max_rows": ("i", "i"),
    "rmlx_postnorm_in": ("ppppfpii" "pppqi" "piiiip", "i"),
    "rmlx_postnorm_gated": ("ppppfpii" "piiifip", "i"),
    "rmlx_matvec_out": ("ppipiiiiip", "i"),
})


def pad_to(n: int, m: int) -> int:
    return (n + m - 1) // m * m


def embed_norm(table: torch.Tensor, ids: torch.Tensor, w: torch.Tensor, eps: float, x: torch.Tensor, h: torch.Tensor,
               pdl: bool = False) -> None:
    """x[t] = RMSNorm(table[ids[t]]) in fp32, h[t] the same in the compute type."""
    _lib.require_cuda_tensor(table, ids, w, x, h)
    assert ids.dtype == torch.int32 and x.dtype == w.dtype == torch.float32 and h.dtype == table.dtype
    assert x.shape == h.shape and x.is_contiguous() and h.is_contiguous() and table.is_contiguous()
    rc = _lib.cuda().rmlx_embed_norm(table.data_ptr(), ids.data_ptr(), w.data_ptr(), eps, x.data_ptr(), h.data_ptr(),
                                     ids.numel(), table.shape[1], x.shape[1], table.shape[0], _f32(table), int(pdl),
                                     _lib.stream_ptr())
    _lib.check(rc, "embed_norm")


def post_norm_add(y: torch.Tensor, w: torch.Tensor, eps: float, width: int, x: torch.Tensor,
                  h: Optional[torch.Tensor], pdl: bool = False) -> None:
    """x += RMSNorm(y) * w on the fp32 residual, h = x in the compute type."""
    _lib.require_cuda_tensor(y, w, x, h)
    t, ldx = x.shape
    assert x.dtype == torch.float32 and x.is_contiguous() and y.shape[0] == t and w.numel() == ldx
    assert h is None or (h.shape == x.shape and h.is_contiguous())
    rc = _lib.cuda().rmlx_post_norm_add(y.data_ptr(), y.stride(0), _f32(y), w.data_ptr(), eps, x.data_ptr(),
                                        _lib.ptr(h), t, width, ldx, 0 if h is None else _f32(h), int(pdl),
                                        _lib.stream_ptr())
    _lib.check(rc, "post_norm_add")


def head_norm_append(raw: torch.Tensor, q_w: torch.Tensor, k_w: torch.Tensor, eps: float, q: torch.Tensor,
                     k_cache: torch.Tensor, v_cache: torch.Tensor, block_table: torch.Tensor, positions: torch.Tensor,
                     token_seq: Optional[torch.Tensor], heads: int, dim: int, vdim: int, pdl: bool = False) -> None:
    """Per-head RMS norm of queries and keys (weights [dim]); queries to ``q``, keys / values to their pages."""
    _lib.require_cuda_tensor(raw, q, k_cache, v_cache, block_table, positions, token_seq)
    t, hkv = raw.shape[0], k_cache.shape[1]
    assert q.shape == (t, heads, k_cache.shape[3]) and q.dtype == k_cache.dtype == v_cache.dtype
    assert q_w.numel() == k_w.numel() == dim and q_w.dtype == k_w.dtype == torch.float32
    rc = _lib.cuda().rmlx_head_norm_append(
        raw.data_ptr(), raw.stride(0), _f32(raw), q_w.data_ptr(), k_w.data_ptr(), eps, q.data_ptr(), k_cache.data_ptr(),
        v_cache.data_ptr(), block_table.data_ptr(), positions.data_ptr(), _lib.ptr(token_seq), t, heads, hkv, dim, vdim,
        k_cache.shape[3], v_cache.shape[3], block_table.stride(0), k_cache.shape[2], _f32(q), int(pdl), _lib.stream_ptr())
    _lib.check(rc, "head_norm_append")


def latent_append(q_raw: torch.Tensor, down: Optional[torch.Tensor], c_w: Optional[torch.Tensor], eps: float,
                  inv_freq: torch.Tensor, q: torch.Tensor, q_abs: Optional[torch.Tensor], cache: torch.Tensor,
                  block_table: torch.Tensor, positions: torch.Tensor, token_seq: Optional[torch.Tensor], heads: int,
                  dim: int, rot: int, rank: int, dim_p: int, rot_p: int, lat_p: int, pdl: bool = False) -> None:
    """Rotated queries of ``q_raw`` [T, H * (dim + rot)] to ``q`` [T, H, dim_p + rot_p] (their rotated part also
    behind the latent part of ``q_abs`` [T, H, lat_p + rot_p]); of ``down`` [T, latent | key part] the normed
    latent and the rotated key part to the token's cache row (None: the row is another layer's and in place).
    ``inv_freq`` fp32 [rotated pairs]."""
    _lib.require_cuda_tensor(q_raw, down, c_w, inv_freq, q, q_abs, cache, block_table, positions, token_seq)
    t = q_raw.shape[0]
    assert q.shape == (t, heads, dim_p + rot_p) and q.is_contiguous() and q.dtype == cache.dtype
    assert q_abs is None or (q_abs.shape == (t, heads, lat_p + rot_p) and q_abs.is_contiguous())
    assert cache.shape[1] == 1 and (down is None or (c_w.numel() == rank and down.dtype == q_raw.dtype))
    rc = _lib.cuda().rmlx_latent_append(
        q_raw.data_ptr(), q_raw.stride(0), _lib.ptr(down), 0 if down is None else down.stride(0), _f32(q_raw), _lib.ptr(c_w),
        eps, inv_freq.data_ptr(), 2 * inv_freq.numel(), q.data_ptr(), _lib.ptr(q_abs), cache.data_ptr(), cache.shape[3],
        block_table.data_ptr(), positions.data_ptr(), _lib.ptr(token_seq), t, heads, dim, rot, rank, dim_p, rot_p, lat_p,
        block_table.stride(0), cache.shape[2], _f32(q), int(pdl), _lib.stream_ptr())
    _lib.check(rc, "latent_append")


def head_gemv(w: torch.Tensor, x: torch.Tensor, out: torch.Tensor, rows: Optional[torch.Tensor] = None,
              pdl: bool = False) -> None:
    """out[t, h, :N] = w[h] x[t, h, :K] for the rows given (default: all); w [H, N, K], x and out [T, H, ..]
    (the first K / N values of a head's row)."""
    _lib.require_cuda_tensor(w, x, out, rows)
    hd, n, k = w.shape
    assert w.is_contiguous() and x.dtype == out.dtype == w.dtype and x.shape[1] == out.shape[1] == hd
    assert x.shape[2] >= k and out.shape[2] >= n and x.stride(2) == out.stride(2) == 1
    rc = _lib.cuda().rmlx_head_gemv(w.data_ptr(), x.data_ptr(), x.stride(0), x.stride(1), out.data_ptr(), out.stride(0),
                                    out.stride(1), _lib.ptr(rows), x.shape[0] if rows is None else rows.numel(), hd, n, k,
                                    _f32(w), int(pdl), _lib.stream_ptr())
    _lib.check(rc, "head_gemv")


def linear(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, pdl: bool = False) -> torch.Tensor:
    """out = x w^T in the activations' type (bf16: tcgen05 GEMM, fp32: FFMA)."""
    if not _f32(x):
        return gemm_bf16(x, w, out=out, pdl=pdl)
    _lib.require_cuda_tensor(x, w, out)
    assert out.shape == (x.shape[0], w.shape[0]) and x.shape[1] == w.shape[1]
    rc = _lib.cuda().rmlx_sgemm(x.data_ptr(), x.stride(0), w.data_ptr(), w.stride(0), out.data_ptr(), out.stride(0),
                                x.shape[0], w.shape[0], x.shape[1], int(pdl), _lib.stream_ptr())
    _lib.check(rc, "sgemm")
    return out


def gated_act(gu: torch.Tensor, out: torch.Tensor, limit: float = 0.0, pdl: bool = False) -> torch.Tensor:
    """out = act(gate, up) of rows [gate | up] (csrc/common/gated.cuh)."""
    _lib.require_cuda_tensor(gu, out)
    assert gu.is_contiguous() and out.is_contiguous() and gu.shape[1] == 2 * out.shape[1] and gu.dtype == out.dtype
    rc = _lib.cuda().rmlx_gated_act(gu.data_ptr(), out.data_ptr(), out.shape[0], out.shape[1], limit, _f32(gu), int(pdl),
                                    _lib.stream_ptr())
    _lib.check(rc, "gated_act")
    return out


def gated_linear(x: torch.Tensor, w: LinearWeight, limit: float, act: torch.Tensor, scratch: Optional[torch.Tensor],
                 pdl: bool = False) -> torch.Tensor:
    """act = gated activation of x w^T, w = [gate; up]. bf16: in the GEMM's epilogue; fp32: through ``scratch``
    [T, 2 n]."""
    if not _f32(x):
        return xgemm(x, w, out=act, swiglu=True, gate_limit=limit, pdl=pdl)
    linear(x, w.w, scratch, pdl=pdl)
    return gated_act(scratch, act, limit, pdl=pdl)


def tanh_rows(x: torch.Tensor, out: torch.Tensor, pdl: bool = False) -> torch.Tensor:
    _lib.require_cuda_tensor(x, out)
    assert x.dtype == torch.float32 and x.is_contiguous() and out.is_contiguous() and x.numel() == out.numel()
    rc = _lib.cuda().rmlx_tanh_rows(x.data_ptr(), out.data_ptr(), x.numel(), _f32(out), int(pdl), _lib.stream_ptr())
    _lib.check(rc, "tanh_rows")
    return out


# ------------------------------------------------------------------ decode projections (csrc/kernels/postnorm_gemv.cu)
def max_rows(k: int) -> int:
    """Rows one launch of the decode projections takes for ``k`` staged values (0: none)."""
    return int(_lib.cuda().rmlx_postnorm_max_rows(k))


def _chunks(b: int, k: int):
    step = max_rows(k)
    if step < 1:
        raise _lib.NativeError(f"decode projections: {k} values do not fit a block's shared memory")
    return [(lo, min(b, lo + step)) for lo in range(0, b, step)]


@dataclass
class Pending:
    """A finished sublayer's output that still has to be normed and added to the residual: what the next kernel
    that reads the residual does on the way."""
    y: Optional[torch.Tensor]        # fp32 [B, width_p]; None: nothing pending
    w: Optional[torch.Tensor]        # fp32 [width_p]


def postnorm_in(x: torch.Tensor, pending: Pending, eps: float, width: int, x_out: torch.Tensor, w: torch.Tensor,
                out: torch.Tensor, shift=None, pdl: bool = False) -> None:
    """x_out = x + RMSNorm(pending); out = W x_out in fp32. ``shift``: (mu [5, width_p], prev [slots, width_p],
    slots, segment rows) - the row segments of W then read their token-shift mixes of x_out."""
    _lib.require_cuda_tensor(x, x_out, w, out, pending.y)
    b, k = x.shape
    assert x.dtype == x_out.dtype == out.dtype == torch.float32 and w.dtype == torch.bfloat16 and w.is_contiguous()
    assert w.shape[1] == k and x.is_contiguous() and x_out.is_contiguous() and out.shape[0] == b
    for lo, hi in _chunks(b, k):
        y = None if pending.y is None else pending.y[lo:].data_ptr()
        sh = (None, None, None, 0, 0) if shift is None else (
            shift[0].data_ptr(), shift[1].data_ptr(), shift[2][lo:].data_ptr(), shift[1].stride(0), shift[3])
        rc = _lib.cuda().rmlx_postnorm_in(w.data_ptr(), x[lo:].data_ptr(), y, _lib.ptr(pending.w), eps, x_out[lo:].data_ptr(),
                                          width, k, *sh, out[lo:].data_ptr(), out.stride(0), hi - lo, w.shape[0], int(pdl),
                                          _lib.stream_ptr())
        _lib.check(rc, "postnorm_in")


def postnorm_gated(x: torch.Tensor, pending: Pending, eps: float, width: int, x_out: torch.Tensor, w: torch.Tensor,
                   limit: float, act: torch.Tensor, pdl: bool = False) -> None:
    """x_out = x + RMSNorm(pending); act = gated activation of W x_out, W = [gate; up]."""
    _lib.require_cuda_tensor(x, x_out, w, act, pending.y)
    b, k = x.shape
    assert w.shape == (2 * act.shape[1], k) and w.is_contiguous() and act.dtype == w.dtype == torch.bfloat16
    for lo, hi in _chunks(b, k):
        y = None if pending.y is None else pending.y[lo:].data_ptr()
        rc = _lib.cuda().rmlx_postnorm_gated(w.data_ptr(), x[lo:].data_ptr(), y, _lib.ptr(pending.w), eps,
                                             x_out[lo:].data_ptr(), width, k, act[lo:].data_ptr(), act.stride(0), hi - lo,
                                             act.shape[1], limit, int(pdl), _lib.stream_ptr())
        _lib.check(rc, "postnorm_gated")


def rows_in(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, pdl: bool = False) -> torch.Tensor:
    """out = x w^T of a few finished fp32 rows (``postnorm_in`` with nothing pending)."""
    _lib.require_cuda_tensor(x, w, out)
    b, k = x.shape
    assert x.dtype == out.dtype == torch.float32 and w.dtype == torch.bfloat16 and w.is_contiguous() and w.shape[1] == k
    assert x.is_contiguous() and out.shape == (b, w.shape[0])
    for lo, hi in _chunks(b, k):
        rc = _lib.cuda().rmlx_postnorm_in(w.data_ptr(), x[lo:].data_ptr(), None, None, 0.0, None, k, k, None, None, None, 0, 0,
                                          out[lo:].data_ptr(), out.stride(0), hi - lo, w.shape[0], int(pdl), _lib.stream_ptr())
        _lib.check(rc, "postnorm_in")
    return out


def matvec_out(a: torch.Tensor, w: torch.Tensor, y: torch.Tensor, pdl: bool = False) -> torch.Tensor:
    """y = a w^T, bf16 in, fp32 out, a few rows."""
    _lib.require_cuda_tensor(a, w, y)
    b, k = a.shape
    assert a.dtype == w.dtype == torch.bfloat16 and y.dtype == torch.float32 and w.is_contiguous() and w.shape[1] == k
    for lo, hi in _chunks(b, k):
        rc = _lib.cuda().rmlx_matvec_out(w.data_ptr(), a[lo:].data_ptr(), a.stride(0), y[lo:].data_ptr(), y.stride(0), hi - lo,
                                         w.shape[0], k, int(pdl), _lib.stream_ptr())
        _lib.check(rc, "matvec_out")
    return y
