"""Row operations of decoders with a layer norm before and after each sublayer and a short convolution over what a sublayer
reads (csrc/kernels/sandwich_rows.cu), and their decode projections (sandwich_gemv.cu). Activations are bf16 or fp32; the
dtype of the tensors picks the kernels. A norm's weight and bias are one fp32 tensor [2, row width]."""
from __future__ import annotations

import functools
from typing import Optional, Tuple

import torch

from .. import _lib
from .parallel_block import _f32
from .post_norm import _chunks
from .routed import Routing

_lib.register_cuda_sigs({
    "rmlx_sandwich_norm": ("ppippi" "pppf" "iiiiip", "i"),
    "rmlx_short_conv": ("ppipi" "pq" "ppiiiip", "i"),
    "rmlx_poly_norm": ("ppfp" "iiiiip", "i"),
    "rmlx_sandwich_step_max_width": ("", "i"),
    "rmlx_sandwich_step": ("ppi" "ppi" "pppi" "pi" "pqp" "fiiiip", "i"),
    "rmlx_lightning_step": ("piii" "ppp" "q" "pi" "iiii" "iip", "i"),
    "rmlx_poly_out": ("ppipfpi" "iiiiip", "i"),
    "rmlx_gated_out": ("ppipipfpi" "iiiiip", "i"),
})


def _affine_ok(w: Optional[torch.Tensor], ld: int) -> bool:
    return w is None or (w.dtype == torch.float32 and w.is_contiguous() and w.shape == (2, ld))


def sandwich_norm(x: torch.Tensor, y: Optional[torch.Tensor], wy: Optional[torch.Tensor], wh: Optional[torch.Tensor],
                  h: Optional[torch.Tensor], eps: float, width: int, routing: Optional[Routing] = None, pdl: bool = False) -> None:
    """x += LN(y; wy), h = LN(x; wh) on the fp32 residual; y may be None (nothing is added) or, with ``routing``, the rows of
    the tokens' experts; h may be None."""
    _lib.require_cuda_tensor(x, y, wy, wh, h)
    t, ldx = x.shape
    ref = h if h is not None else y
    assert x.dtype == torch.float32 and x.is_contiguous() and _affine_ok(wy, ldx) and _affine_ok(wh, ldx)
    assert h is None or (h.shape == x.shape and h.is_contiguous())
    assert y is None or (y.dtype == ref.dtype and y.stride(1) == 1 and (routing is not None or y.shape[0] == t))
    rc = _lib.cuda().rmlx_sandwich_norm(
        x.data_ptr(), _lib.ptr(y), 0 if y is None else y.stride(0), None if routing is None else routing.row_of_pair.data_ptr(),
        None if routing is None else routing.weights.data_ptr(), 0 if routing is None else routing.idx.shape[1], _lib.ptr(wy),
        _lib.ptr(wh), _lib.ptr(h), eps, t, width, ldx, _f32(ref), int(pdl), _lib.stream_ptr())
    _lib.check(rc, "sandwich_norm")


def _carried_ok(carried: Optional[torch.Tensor], taps: int, ld: int) -> bool:
    return taps == 1 or (carried is not None and carried.dtype == torch.float32 and carried.shape[1:] == (taps - 1, ld) and
                         carried.stride()[1:] == (ld, 1))


def short_conv(h: torch.Tensor, w: torch.Tensor, carried: Optional[torch.Tensor], out: torch.Tensor, slots: Optional[torch.Tensor],
               runs: Optional[torch.Tensor] = None, pdl: bool = False) -> torch.Tensor:
    """out = h + its causal depthwise convolution over every sequence's new tokens (w fp32 [taps, width], oldest first), after
    the inputs ``carried`` [slots, taps - 1, width], which are advanced. ``slots`` int32 [T]: the slot of every row (None: only with one tap); ``runs``
    int32 [n, 4] (first row, rows, slot, -), None: every row its own sequence."""
    _lib.require_cuda_tensor(h, w, carried, out, slots, runs)
    t, ld = h.shape
    taps = w.shape[0]
    assert h.is_contiguous() and out.is_contiguous() and out.shape == h.shape and out.dtype == h.dtype
    assert w.dtype == torch.float32 and w.is_contiguous() and w.shape[1] == ld and _carried_ok(carried, taps, ld)
    assert taps == 1 or slots.numel() == t
    rc = _lib.cuda().rmlx_short_conv(
        h.data_ptr(), out.data_ptr(), ld, w.data_ptr(), taps, _lib.ptr(carried) if taps > 1 else None,
        carried.stride(0) if taps > 1 else 0, _lib.ptr(runs), _lib.ptr(slots), t if runs is None else runs.shape[0], t, _f32(h),
        int(pdl), _lib.stream_ptr())
    _lib.check(rc, "short_conv")
    return out


def poly_norm(z: torch.Tensor, act: torch.Tensor, eps: float, width: int, out: torch.Tensor, pdl: bool = False) -> torch.Tensor:
    """out = a N(z) + b N(z^2) + c N(z^3) + e over the first ``width`` columns (act fp32 [4]), zeros in the rest."""
    _lib.require_cuda_tensor(z, act, out)
    assert z.is_contiguous() and out.is_contiguous() and z.shape == out.shape and z.dtype == out.dtype
    assert act.dtype == torch.float32 and act.numel() == 4
    rc = _lib.cuda().rmlx_poly_norm(z.data_ptr(), act.data_ptr(), eps, out.data_ptr(), z.shape[0], width, z.shape[1], _f32(z),
                                    int(pdl), _lib.stream_ptr())
    _lib.check(rc, "poly_norm")
    return out


# ------------------------------------------------------------------ decode
@functools.lru_cache(maxsize=None)
def step_max_width() -> int:
    return int(_lib.cuda().rmlx_sandwich_step_max_width())


def sandwich_step(x: torch.Tensor, y: Optional[torch.Tensor], wy: Optional[torch.Tensor], wh: torch.Tensor, h: torch.Tensor,
                  eps: float, width: int, conv: Optional[Tuple[torch.Tensor, Optional[torch.Tensor], Optional[torch.Tensor]]] = None,
                  routing: Optional[Routing] = None, pdl: bool = False) -> None:
    """A decode row per sequence: ``sandwich_norm`` and, with ``conv`` (weights, carried inputs, slots), ``short_conv`` in one
    launch: x += LN(y; wy), h = LN(x; wh) + its convolution. x fp32; y and h both fp32 or both bf16."""
    w, carried, slots = conv or (None, None, None)
    _lib.require_cuda_tensor(x, y, wy, wh, h, w, carried, slots)
    b, ldx = x.shape
    assert x.dtype == torch.float32 and x.is_contiguous() and h.is_contiguous() and h.shape == x.shape
    assert _affine_ok(wy, ldx) and _affine_ok(wh, ldx)
    assert y is None or (y.dtype == h.dtype and y.stride(1) == 1 and (routing is not None or y.shape[0] == b))
    taps = 0 if w is None else w.shape[0]
    assert w is None or (w.dtype == torch.float32 and w.is_contiguous() and w.shape[1] == ldx and _carried_ok(carried, taps, ldx))
    rc = _lib.cuda().rmlx_sandwich_step(
        x.data_ptr(), _lib.ptr(y), 0 if y is None else y.stride(0),
        None if routing is None else routing.row_of_pair.data_ptr(), None if routing is None else routing.weights.data_ptr(),
        0 if routing is None else routing.idx.shape[1], _lib.ptr(wy), wh.data_ptr(), h.data_ptr(), _f32(h), _lib.ptr(w), taps,
        _lib.ptr(carried) if taps > 1 else None, carried.stride(0) if taps > 1 else 0, _lib.ptr(slots), eps, b, width, ldx, int(pdl),
        _lib.stream_ptr())
    _lib.check(rc, "sandwich_step")


def poly_out(z: torch.Tensor, act: torch.Tensor, eps: float, width: int, w: torch.Tensor, y: torch.Tensor, pdl: bool = False) -> None:
    """y = W poly_norm(z), z fp32 [B, K] with ``width`` real columns, W bf16 [N, K] (zero from ``width`` on)."""
    _lib.require_cuda_tensor(z, act, w, y)
    n, k = w.shape
    assert z.dtype == y.dtype == torch.float32 and w.dtype == torch.bfloat16 and w.is_contiguous() and z.shape[1] >= k
    for lo, hi in _chunks(z.shape[0], k):
        rc = _lib.cuda().rmlx_poly_out(w.data_ptr(), z[lo:].data_ptr(), z.stride(0), act.data_ptr(), eps, y[lo:].data_ptr(),
                                       y.stride(0), hi - lo, n, k, width, int(pdl), _lib.stream_ptr())
        _lib.check(rc, "poly_out")


def gated_out(o: torch.Tensor, gate: torch.Tensor, norm: torch.Tensor, eps: float, w: torch.Tensor, y: torch.Tensor,
              pdl: bool = False) -> None:
    """y = W (o / rms(o) * norm * sigmoid(gate)) over the first ``norm.numel()`` columns; o, gate fp32 [B, >= K]."""
    _lib.require_cuda_tensor(o, gate, norm, w, y)
    n, k = w.shape
    assert o.dtype == gate.dtype == y.dtype == norm.dtype == torch.float32 and w.dtype == torch.bfloat16 and w.is_contiguous()
    for lo, hi in _chunks(o.shape[0], k):
        rc = _lib.cuda().rmlx_gated_out(w.data_ptr(), o[lo:].data_ptr(), o.stride(0), gate[lo:].data_ptr(), gate.stride(0),
                                        norm.data_ptr(), eps, y[lo:].data_ptr(), y.stride(0), hi - lo, n, k, norm.numel(), int(pdl),
                                        _lib.stream_ptr())
        _lib.check(rc, "gated_out")


def lightning_step(raw: torch.Tensor, at_k: int, at_v: int, decay: torch.Tensor, slots: torch.Tensor, state: torch.Tensor,
                   out: torch.Tensor, pdl: bool = False) -> None:
    """One token per row of ``scan.lightning_scan``: raw fp32 or bf16 [B, ..] = q at 0, k and v at their columns; out fp32 [B, >= H vdim]."""
    _lib.require_cuda_tensor(raw, decay, slots, state, out)
    _, h, n, d = state.shape
    assert out.dtype == decay.dtype == torch.float32 and state.stride()[1:] == (n * d, d, 1)
    assert slots.dtype == torch.int32 and decay.numel() == h
    rc = _lib.cuda().rmlx_lightning_step(
        raw.data_ptr(), raw.stride(0), at_k, at_v, decay.data_ptr(), slots.data_ptr(), state.data_ptr(), state.stride(0),
        out.data_ptr(), out.stride(0), raw.shape[0], h, n, d, _f32(raw), int(pdl), _lib.stream_ptr())
    _lib.check(rc, "lightning_step")
