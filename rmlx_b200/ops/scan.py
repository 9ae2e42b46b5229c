"""Linear recurrences token by token (csrc/kernels/linear_scan.cu): gated linear attention, state-space heads with
their short convolution, lightning attention, and the norm of their outputs with a gate; the first two's decode steps
(twin_norm_gemv.cu). A sequence's state is its slot's row of a
flat fp32 pool (``PagedKvCache.layer_state`` views)."""
from __future__ import annotations

from typing import Optional

import torch

from .. import _lib
from .gemm import GemmStatus
from .parallel_block import _f32

SCAN_MAX_ROWS = 256          # rows of a state (key channels)

_lib.register_cuda_sigs({
    "rmlx_scan_max_rows": ("", "i"),
    "rmlx_scan_record": ("iiii", "q"),
    "rmlx_gla_scan": ("pppi" "pip" "ff" "pippi" "pqpi" "iiii" "pip", "i"),
    "rmlx_ssd_scan": ("piii" "ppi" "pppp" "pippi" "pqpi" "iiiii" "pip", "i"),
    "rmlx_gla_decode_supported": ("ii", "i"),
    "rmlx_gla_decode": ("piiiii" "pipff" "pfp" "pq" "pi" "iiiiip", "i"),
    "rmlx_ssd_decode": ("piii" "ppi" "ppppp" "pq" "pi" "pfi" "pi" "iiiii" "ip", "i"),
    "rmlx_lightning_scan": ("pppip" "pippi" "pqpi" "iiii" "pip", "i"),
    "rmlx_gated_norm": ("pipipfpi" "iiiiiiip", "i"),
})


def record(n: int, d: int, one: bool = False, per: int = 1) -> int:
    """Scratch floats per row and head of a state [n, d]; ``one``: heads with a single decay, ``per`` of which
    share their keys and queries."""
    return int(_lib.cuda().rmlx_scan_record(n, d, int(one), per))


def _segments(runs: Optional[torch.Tensor], slots: Optional[torch.Tensor]) -> int:
    return runs.shape[0] if runs is not None else slots.numel()


def gla_scan(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, z: torch.Tensor, bias: torch.Tensor, tau: float, scale: float,
             state: torch.Tensor, out: torch.Tensor, rec: torch.Tensor, runs: Optional[torch.Tensor] = None,
             slots: Optional[torch.Tensor] = None, pdl: bool = False) -> None:
    """S <- diag(sigmoid(z + bias)^(1 / tau)) S + k v^T, out = S^T (q * scale) for every sequence's new tokens on top of
    ``state`` [slots, H, dim, vdim]. q, k, v [T, ..] in the compute type with one row stride, z and out fp32, ``rec``
    scratch of T * H * ``record(dim, vdim)`` floats. ``runs`` int32 [n, 4] (first row, rows, slot, -), or ``slots``:
    every row its own sequence."""
    _lib.require_cuda_tensor(q, k, v, z, bias, state, out, rec, runs, slots)
    _, h, n, d = state.shape
    t = q.shape[0]
    assert q.stride(0) == k.stride(0) == v.stride(0) and q.dtype == k.dtype == v.dtype
    assert z.dtype == bias.dtype == out.dtype == state.dtype == torch.float32 and state.stride()[1:] == (n * d, d, 1)
    assert bias.numel() == h * n and rec.is_contiguous() and rec.numel() >= t * h * record(n, d)
    rc = _lib.cuda().rmlx_gla_scan(
        q.data_ptr(), k.data_ptr(), v.data_ptr(), q.stride(0), z.data_ptr(), z.stride(0), bias.data_ptr(), 1.0 / tau, scale,
        rec.data_ptr(), t, _lib.ptr(runs), _lib.ptr(slots), _segments(runs, slots), state.data_ptr(), state.stride(0),
        out.data_ptr(), out.stride(0), h, n, d, _f32(q), GemmStatus.get(q.device).data_ptr(), int(pdl), _lib.stream_ptr())
    _lib.check(rc, "gla_scan")


def ssd_scan(raw: torch.Tensor, x_at: int, dt_at: int, conv_w: torch.Tensor, conv_b: torch.Tensor,
             carried: Optional[torch.Tensor], dt_bias: torch.Tensor, a_log: torch.Tensor, skip: torch.Tensor, groups: int,
             state: torch.Tensor, out: torch.Tensor, rec: torch.Tensor, row_slots: torch.Tensor,
             runs: Optional[torch.Tensor] = None, pdl: bool = False) -> None:
    """State-space heads over raw [T, ..] = x | B | C at column ``x_at``, dt at ``dt_at``: convolution (``conv_w`` fp32
    [taps, channels], oldest first) with silu, dt = softplus(dt + dt_bias), S <- exp(-exp(a_log) dt) S + dt B x^T, out =
    S^T C + skip x. ``carried`` [slots, taps - 1, channels] and ``state`` [slots, H, n, d] are advanced; ``row_slots``
    int32 [T]; ``runs`` as in ``gla_scan`` (None: every row its own sequence)."""
    _lib.require_cuda_tensor(raw, conv_w, conv_b, dt_bias, a_log, skip, state, out, rec, row_slots, runs)
    _, h, n, d = state.shape
    t, (taps, ch) = raw.shape[0], conv_w.shape
    assert ch == conv_b.numel() == h * d + 2 * groups * n and h % groups == 0 and conv_w.is_contiguous()
    assert conv_w.dtype == conv_b.dtype == dt_bias.dtype == a_log.dtype == skip.dtype == out.dtype == torch.float32
    assert state.stride()[1:] == (n * d, d, 1) and dt_bias.numel() == a_log.numel() == skip.numel() == h
    assert taps == 1 or (carried.shape[1:] == (taps - 1, ch) and carried.stride()[1:] == (ch, 1) and
                         carried.stride(0) == state.stride(0))
    assert row_slots.numel() == t and rec.is_contiguous() and rec.numel() >= t * h * record(n, d, True, h // groups)
    rc = _lib.cuda().rmlx_ssd_scan(
        raw.data_ptr(), raw.stride(0), x_at, dt_at, conv_w.data_ptr(), conv_b.data_ptr(), taps,
        carried.data_ptr() if taps > 1 else None, dt_bias.data_ptr(), a_log.data_ptr(), skip.data_ptr(), rec.data_ptr(), t,
        _lib.ptr(runs), row_slots.data_ptr(), _segments(runs, row_slots), state.data_ptr(), state.stride(0), out.data_ptr(),
        out.stride(0), h, groups, n, d, _f32(raw), GemmStatus.get(raw.device).data_ptr(), int(pdl), _lib.stream_ptr())
    _lib.check(rc, "ssd_scan")


def lightning_scan(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor, state: torch.Tensor, out: torch.Tensor,
                   rec: torch.Tensor, runs: Optional[torch.Tensor] = None, slots: Optional[torch.Tensor] = None,
                   pdl: bool = False) -> None:
    """S <- decay S + silu(k) silu(v)^T, out = S^T silu(q) with one constant decay per head (fp32 [H]); ``rec``: scratch of
    T * H * ``record(dim, vdim, True)`` floats, the rest as in ``gla_scan``."""
    _lib.require_cuda_tensor(q, k, v, decay, state, out, rec, runs, slots)
    _, h, n, d = state.shape
    t = q.shape[0]
    assert q.stride(0) == k.stride(0) == v.stride(0) and q.dtype == k.dtype == v.dtype
    assert decay.dtype == out.dtype == state.dtype == torch.float32 and state.stride()[1:] == (n * d, d, 1)
    assert decay.numel() == h and rec.is_contiguous() and rec.numel() >= t * h * record(n, d, True)
    rc = _lib.cuda().rmlx_lightning_scan(
        q.data_ptr(), k.data_ptr(), v.data_ptr(), q.stride(0), decay.data_ptr(), rec.data_ptr(), t, _lib.ptr(runs), _lib.ptr(slots),
        _segments(runs, slots), state.data_ptr(), state.stride(0), out.data_ptr(), out.stride(0), h, n, d, _f32(q),
        GemmStatus.get(q.device).data_ptr(), int(pdl), _lib.stream_ptr())
    _lib.check(rc, "lightning_scan")


def gated_norm(o: torch.Tensor, gate: torch.Tensor, w: torch.Tensor, eps: float, groups: int, out: torch.Tensor,
               gate_first: bool, sigmoid: bool = False, pdl: bool = False) -> torch.Tensor:
    """RMS norm of the first ``w.numel()`` columns in ``groups`` equal parts, times w, with silu(gate) (``sigmoid``:
    sigmoid(gate)) multiplied before (``gate_first``) or after the norm."""
    _lib.require_cuda_tensor(o, gate, w, out)
    assert o.dtype == w.dtype == torch.float32 and gate.dtype == out.dtype and w.numel() % groups == 0
    rc = _lib.cuda().rmlx_gated_norm(o.data_ptr(), o.stride(0), gate.data_ptr(), gate.stride(0), w.data_ptr(), eps,
                                     out.data_ptr(), out.stride(0), o.shape[0], groups, w.numel() // groups, int(gate_first),
                                     int(sigmoid), _f32(out), int(pdl), _lib.stream_ptr())
    _lib.check(rc, "gated_norm")
    return out


# ------------------------------------------------------------------ decode (csrc/kernels/twin_norm_gemv.cu)
def gla_decode_supported(n: int, d: int) -> bool:
    return bool(_lib.cuda().rmlx_gla_decode_supported(n, d))


def gla_decode(raw: torch.Tensor, at, a2: torch.Tensor, bias: torch.Tensor, tau: float, scale: float, norm: torch.Tensor,
               eps: float, slots: torch.Tensor, state: torch.Tensor, out: torch.Tensor, pdl: bool = False) -> None:
    """One token per row through decay, state, head norm and gate: raw fp32 [B, ..] with q, k, v, g and the decay's first
    factor at the columns ``at``, ``a2`` bf16 [>= H dim, rank]; out bf16 [B, >= H vdim]."""
    _lib.require_cuda_tensor(raw, a2, bias, norm, slots, state, out)
    _, h, n, d = state.shape
    assert raw.dtype == torch.float32 and a2.dtype == out.dtype == torch.bfloat16 and a2.is_contiguous() and at[0] == 0
    assert state.stride()[1:] == (n * d, d, 1) and slots.dtype == torch.int32 and bias.numel() == h * n and norm.numel() == h * d
    rc = _lib.cuda().rmlx_gla_decode(
        raw.data_ptr(), raw.stride(0), at[1], at[2], at[3], at[4], a2.data_ptr(), a2.shape[1], bias.data_ptr(), 1.0 / tau, scale,
        norm.data_ptr(), eps, slots.data_ptr(), state.data_ptr(), state.stride(0), out.data_ptr(), out.stride(0), raw.shape[0], h,
        n, d, int(pdl), _lib.stream_ptr())
    _lib.check(rc, "gla_decode")


def ssd_decode(raw: torch.Tensor, x_at: int, dt_at: int, conv_w: torch.Tensor, conv_b: torch.Tensor,
               carried: Optional[torch.Tensor], dt_bias: torch.Tensor, a_log: torch.Tensor, skip: torch.Tensor, groups: int,
               slots: torch.Tensor, state: torch.Tensor, y: torch.Tensor, norm: torch.Tensor, eps: float, norm_groups: int,
               out: torch.Tensor, pdl: bool = False) -> None:
    """One token per row through convolution, state, gate and grouped norm: raw fp32 [B, ..] = z at 0, x | B | C at
    ``x_at``, dt at ``dt_at``; ``y`` fp32 scratch [B, >= H d], out bf16 [B, >= H d]."""
    _lib.require_cuda_tensor(raw, conv_w, conv_b, dt_bias, a_log, skip, slots, state, y, norm, out)
    _, h, n, d = state.shape
    taps, ch = conv_w.shape
    assert raw.dtype == y.dtype == torch.float32 and out.dtype == torch.bfloat16 and ch == h * d + 2 * groups * n
    assert state.stride()[1:] == (n * d, d, 1) and slots.dtype == torch.int32 and norm.numel() == h * d
    assert taps == 1 or (carried.shape[1:] == (taps - 1, ch) and carried.stride(0) == state.stride(0))
    rc = _lib.cuda().rmlx_ssd_decode(
        raw.data_ptr(), raw.stride(0), x_at, dt_at, conv_w.data_ptr(), conv_b.data_ptr(), taps,
        carried.data_ptr() if taps > 1 else None, dt_bias.data_ptr(), a_log.data_ptr(), skip.data_ptr(), slots.data_ptr(),
        state.data_ptr(), state.stride(0), y.data_ptr(), y.stride(0), norm.data_ptr(), eps, norm_groups, out.data_ptr(),
        out.stride(0), raw.shape[0], h, groups, n, d, int(pdl), _lib.stream_ptr())
    _lib.check(rc, "ssd_decode")
