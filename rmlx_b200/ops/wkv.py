"""RWKV-style time mixing (csrc/kernels/wkv.cu): token shift, the WKV recurrence and the gated head norm.
A sequence's state is its slot's row of a flat fp32 pool (``PagedKvCache.layer_state`` views)."""
from __future__ import annotations

from typing import Optional

import torch

from .. import _lib
from .gemm import GemmStatus
from .parallel_block import _f32

SHIFT_PARTS = ("r", "k", "v", "g", "w")

_lib.register_cuda_sigs({
    "rmlx_wkv_max_dim": ("", "i"),
    "rmlx_token_shift": ("pippqpipiiip", "i"),
    "rmlx_wkv_record": ("i", "i"),
    "rmlx_wkv_scan": ("pppipippp" "ippi" "ppqpipi" "iiipip", "i"),
    "rmlx_wkv_decode": ("piipipppfp" "ppqpipiiiiip", "i"),
    "rmlx_wkv_finish": ("pipipfpiiiiiip", "i"),
})

WKV_MAX_DIM = 256        # of the recurrence kernel


def token_shift(x: torch.Tensor, mu: torch.Tensor, prev: torch.Tensor, slots: torch.Tensor, each_row: bool,
                out: torch.Tensor, pdl: bool = False) -> None:
    """out[s, t] = x[t] + (x[t - 1] - x[t]) * mu[s]; the row before a sequence's first row of the batch comes
    from ``prev`` [slots, width] at the row's slot. ``each_row``: every row is another sequence."""
    _lib.require_cuda_tensor(x, mu, prev, slots, out)
    t, ldx = x.shape
    assert x.dtype == mu.dtype == prev.dtype == torch.float32 and x.is_contiguous() and mu.is_contiguous()
    assert mu.shape == (len(SHIFT_PARTS), ldx) and out.shape == (len(SHIFT_PARTS), t, ldx) and out.is_contiguous()
    assert prev.shape[1] == ldx and prev.stride(1) == 1 and slots.dtype == torch.int32
    rc = _lib.cuda().rmlx_token_shift(x.data_ptr(), ldx, mu.data_ptr(), prev.data_ptr(), prev.stride(0),
                                      slots.data_ptr(), int(each_row), out.data_ptr(), t, _f32(out), int(pdl),
                                      _lib.stream_ptr())
    _lib.check(rc, "token_shift")


def record(dim: int) -> int:
    """Scratch floats of ``wkv_scan`` per row and head."""
    return int(_lib.cuda().rmlx_wkv_record(dim))


def wkv_scan(r: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor, w0: torch.Tensor, u: torch.Tensor,
             state: torch.Tensor, prev: torch.Tensor, x: torch.Tensor, out: torch.Tensor, rec: torch.Tensor,
             runs: Optional[torch.Tensor] = None, slots: Optional[torch.Tensor] = None, pdl: bool = False) -> None:
    """Runs every sequence's new tokens through the recurrence on top of ``state`` [slots, H, d, d] and
    leaves the new state (and in ``prev`` the last row of ``x``) behind. r, k, v [T, >= H d] in the compute type,
    ``decay`` fp32 logits (w = exp(-exp(decay + w0))), out fp32, ``rec`` scratch of T * H * ``record(d)`` floats.
    ``runs`` int32 [n, 4] (first row, rows, slot, -), or ``slots``: every row its own sequence."""
    _lib.require_cuda_tensor(r, k, v, decay, w0, u, state, prev, x, out, runs, slots)
    _, h, d, _ = state.shape
    assert r.stride(0) == k.stride(0) == v.stride(0) and r.dtype == k.dtype == v.dtype
    assert decay.dtype == out.dtype == x.dtype == state.dtype == torch.float32 and state.stride()[1:] == (d * d, d, 1)
    assert w0.numel() == u.numel() == h * d and state.stride(0) == prev.stride(0)
    n, t = runs.shape[0] if runs is not None else slots.numel(), r.shape[0]
    assert rec.dtype == torch.float32 and rec.is_contiguous() and rec.numel() >= t * h * record(d)
    rc = _lib.cuda().rmlx_wkv_scan(
        r.data_ptr(), k.data_ptr(), v.data_ptr(), r.stride(0), decay.data_ptr(), decay.stride(0), w0.data_ptr(),
        u.data_ptr(), rec.data_ptr(), t, _lib.ptr(runs), _lib.ptr(slots), n, state.data_ptr(), prev.data_ptr(),
        state.stride(0), x.data_ptr(), x.stride(0), out.data_ptr(), out.stride(0), h, d, _f32(r),
        GemmStatus.get(r.device).data_ptr(), int(pdl), _lib.stream_ptr())
    _lib.check(rc, "wkv_scan")


def wkv_finish(o: torch.Tensor, gate: torch.Tensor, norm: torch.Tensor, eps: float, heads: int, dim: int,
               out: torch.Tensor, pdl: bool = False) -> None:
    """out = o / rms(o per head) * norm * silu(gate)."""
    _lib.require_cuda_tensor(o, gate, norm, out)
    assert o.dtype == norm.dtype == torch.float32 and gate.dtype == out.dtype and norm.numel() == heads * dim
    rc = _lib.cuda().rmlx_wkv_finish(o.data_ptr(), o.stride(0), gate.data_ptr(), gate.stride(0), norm.data_ptr(), eps,
                                     out.data_ptr(), out.stride(0), o.shape[0], heads, dim, _f32(out), int(pdl),
                                     _lib.stream_ptr())
    _lib.check(rc, "wkv_finish")


def wkv_decode(raw: torch.Tensor, inner: int, w2: torch.Tensor, w0: torch.Tensor, u: torch.Tensor, norm: torch.Tensor,
               eps: float, slots: torch.Tensor, state: torch.Tensor, prev: torch.Tensor, x: torch.Tensor,
               out: torch.Tensor, pdl: bool = False) -> None:
    """One token per row through recurrence, head norm and gate: raw fp32 [B, 4 * inner + rank] = r | k | v | g | decay
    rank, ``x`` the rows the layer read (kept in ``prev``); out bf16 [B, >= H d] (csrc/kernels/postnorm_gemv.cu)."""
    _lib.require_cuda_tensor(raw, w2, w0, u, norm, slots, state, prev, x, out)
    _, h, d, _ = state.shape
    assert raw.dtype == x.dtype == torch.float32 and w2.dtype == out.dtype == torch.bfloat16 and w2.is_contiguous()
    assert state.stride()[1:] == (d * d, d, 1) and state.stride(0) == prev.stride(0) and slots.dtype == torch.int32
    rc = _lib.cuda().rmlx_wkv_decode(
        raw.data_ptr(), raw.stride(0), inner, w2.data_ptr(), w2.shape[1], w0.data_ptr(), u.data_ptr(), norm.data_ptr(), eps,
        slots.data_ptr(), state.data_ptr(), prev.data_ptr(), state.stride(0), x.data_ptr(), x.stride(0), out.data_ptr(),
        out.stride(0), raw.shape[0], h, d, int(pdl), _lib.stream_ptr())
    _lib.check(rc, "wkv_decode")
