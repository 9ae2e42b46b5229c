"""Row operations of decoders whose mixer and feed-forward read the same residual row through norms of their own
(csrc/kernels/twin_norm_rows.cu), and the decode projections that read it (twin_norm_gemv.cu). Activations are bf16 or fp32; the dtype of the tensors picks the kernels."""
from __future__ import annotations

import math
from typing import Optional, Tuple

import torch

from .. import _lib
from .parallel_block import _f32
from .routed import Routing

_lib.register_cuda_sigs({
    "rmlx_twin_norm": ("ppippi" "ppppf" "iiiiip", "i"),
    "rmlx_rows_norm": ("piipfpi" "iiiip", "i"),
    "rmlx_twin_in_max_rows": ("i", "i"),
    "rmlx_twin_in_gated": ("pppfii" "pipi" "pipif" "iip", "i"),
    "rmlx_twin_in_router": ("pppfii" "pipi" "ppipp" "ppip" "iip", "i"),
    "rmlx_rotary_norm_append": ("piippiff" "ppp" "ppp" "iiiiiiiii" "iii" "iip", "i"),
})


def rotary_frequencies(base: float, dims: int, scaling: Optional[dict] = None) -> Tuple[torch.Tensor, float]:
    """(angle per position of every pair, fp64 [dims / 2]; factor of cos and sin). ``scaling``: YaRN (factor, original,
    fast, slow) - pairs that turn more than ``fast`` times over ``original`` positions keep their speed, those below
    ``slow`` turns are slowed by ``factor``, with a ramp over the pairs between - or Llama's (factor, original, high, low):
    the same by ``high`` and ``low`` turns, with a ramp over the turns and no factor of cos and sin."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = base ** (-2.0 * i / max(dims, 1))
    if not scaling:
        return f, 1.0
    if "high" in scaling:
        turns = scaling["original"] * f / (2 * math.pi)
        s = (turns - scaling["low"]) / (scaling["high"] - scaling["low"])
        mixed = (1 - s) * f / scaling["factor"] + s * f
        slow = torch.where(turns < scaling["low"], f / scaling["factor"], mixed)
        return torch.where(turns > scaling["high"], f, slow), 1.0
    def dim_of(turns):
        return dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo = max(math.floor(dim_of(scaling["fast"])), 0)
    hi = min(math.ceil(dim_of(scaling["slow"])), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return f / scaling["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(scaling["factor"]) + 1.0


def twin_norm(x: torch.Tensor, w1: Optional[torch.Tensor], h1: Optional[torch.Tensor], w2: Optional[torch.Tensor],
              h2: Optional[torch.Tensor], eps: float, width: int, experts: Optional[Tuple[torch.Tensor, Routing]] = None,
              pdl: bool = False) -> None:
    """x += the weighted expert rows (``experts``: rows and their routing), h1 = RMSNorm(x) * w1, h2 = RMSNorm(x) * w2
    (each may be None)."""
    _lib.require_cuda_tensor(x, w1, h1, w2, h2)
    t, ldx = x.shape
    assert x.dtype == torch.float32 and x.is_contiguous()
    ref = h1 if h1 is not None else h2 if h2 is not None else experts[0]
    assert all(h is None or (h.shape == x.shape and h.is_contiguous() and h.dtype == ref.dtype) for h in (h1, h2))
    y, r = experts if experts is not None else (None, None)
    assert y is None or y.dtype == ref.dtype
    rc = _lib.cuda().rmlx_twin_norm(
        x.data_ptr(), _lib.ptr(y), 0 if y is None else y.stride(0), None if r is None else r.row_of_pair.data_ptr(),
        None if r is None else r.weights.data_ptr(), 0 if r is None else r.idx.shape[1], _lib.ptr(w1), _lib.ptr(h1),
        _lib.ptr(w2), _lib.ptr(h2), eps, t, width, ldx, _f32(ref), int(pdl), _lib.stream_ptr())
    _lib.check(rc, "twin_norm")


def rows_norm(x: torch.Tensor, w: torch.Tensor, eps: float, width: int, out: torch.Tensor, pdl: bool = False) -> torch.Tensor:
    """out = RMSNorm of the first ``width`` columns of x times w, zeros in the rest of out's columns."""
    _lib.require_cuda_tensor(x, w, out)
    assert w.dtype == torch.float32 and w.numel() >= width and out.is_contiguous() and x.shape[0] == out.shape[0]
    assert x.stride(1) == 1
    rc = _lib.cuda().rmlx_rows_norm(x.data_ptr(), x.stride(0), _f32(x), w.data_ptr(), eps, out.data_ptr(), out.shape[1],
                                    x.shape[0], width, _f32(out), int(pdl), _lib.stream_ptr())
    _lib.check(rc, "rows_norm")
    return out


def rotary_norm_append(raw: torch.Tensor, bias: Optional[torch.Tensor], inv_freq: torch.Tensor, grow: float, eps: float,
                       q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, block_table: torch.Tensor,
                       positions: torch.Tensor, token_seq: Optional[torch.Tensor], heads: int, dim: int, vdim: int,
                       neighbours: bool = False, norm: bool = True, maps: int = 1, pdl: bool = False) -> None:
    """raw [T, q | k | v] + bias: queries and keys rotated (value i with value i + pairs, or (``neighbours``) 2 i with 2 i + 1;
    cos and sin times ``grow``) and (``norm``) divided by their root mean square per head; queries to ``q``, keys / values
    to their pages. ``maps`` 2 (differential attention): query and key heads of two parts of ``dim`` values, q [T, heads, 2,
    ..], cache rows of two keys."""
    _lib.require_cuda_tensor(raw, bias, inv_freq, q, k_cache, v_cache, block_table, positions, token_seq)
    t, hkv = raw.shape[0], k_cache.shape[1]
    dkp = k_cache.shape[3] // maps
    assert q.shape == ((t, heads, dkp) if maps == 1 else (t, heads, maps, dkp)) and q.is_contiguous()
    assert q.dtype == k_cache.dtype == v_cache.dtype
    assert bias is None or (bias.dtype == torch.float32 and bias.numel() >= (heads + hkv) * maps * dim + hkv * vdim)
    rc = _lib.cuda().rmlx_rotary_norm_append(
        raw.data_ptr(), raw.stride(0), _f32(raw), _lib.ptr(bias), inv_freq.data_ptr(), 2 * inv_freq.numel(), grow, eps,
        q.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), block_table.data_ptr(), positions.data_ptr(),
        _lib.ptr(token_seq), t, heads, hkv, dim, vdim, dkp, v_cache.shape[3], block_table.stride(0),
        k_cache.shape[2], int(neighbours), int(norm), maps, _f32(q), int(pdl), _lib.stream_ptr())
    _lib.check(rc, "rotary_norm_append")


# ------------------------------------------------------------------ decode projections (csrc/kernels/twin_norm_gemv.cu)
def _row_chunks(b: int, k: int):
    step = int(_lib.cuda().rmlx_twin_in_max_rows(k))
    if step < 1:
        raise _lib.NativeError(f"decode projections: {k} values do not fit a block's shared memory")
    return [(lo, min(b, lo + step)) for lo in range(0, b, step)]


def _twin_in_checks(x, w1, w, out):
    _lib.require_cuda_tensor(x, w1, w, out)
    assert x.dtype == out.dtype == w1.dtype == torch.float32 and w.dtype == torch.bfloat16 and x.is_contiguous()
    assert w.is_contiguous() and w.shape[1] == x.shape[1] == w1.numel() and out.shape == (x.shape[0], w.shape[0])


def twin_in(x: torch.Tensor, w1: torch.Tensor, eps: float, width: int, w: torch.Tensor, out: torch.Tensor,
            w2: Optional[torch.Tensor] = None, w_gu: Optional[torch.Tensor] = None, act: Optional[torch.Tensor] = None,
            limit: float = 0.0, pdl: bool = False) -> None:
    """out = W RMSNorm(x; w1) in fp32 and, in the same launch, act = the gated activation of W_gu RMSNorm(x; w2) in bf16
    (W_gu = [gate; up]; None: no feed-forward)."""
    _twin_in_checks(x, w1, w, out)
    assert w_gu is None or (w_gu.is_contiguous() and w_gu.shape == (2 * act.shape[1], x.shape[1]) and act.dtype == w_gu.dtype)
    for lo, hi in _row_chunks(*x.shape):
        a = None if act is None else act[lo:]
        rc = _lib.cuda().rmlx_twin_in_gated(
            x[lo:].data_ptr(), w1.data_ptr(), _lib.ptr(w2), eps, width, x.shape[1], w.data_ptr(), w.shape[0], out[lo:].data_ptr(),
            out.stride(0), _lib.ptr(w_gu), 0 if act is None else act.shape[1], _lib.ptr(a), 0 if act is None else act.stride(0),
            limit, hi - lo, int(pdl), _lib.stream_ptr())
        _lib.check(rc, "twin_in_gated")


def twin_in_router(x: torch.Tensor, w1: torch.Tensor, eps: float, width: int, w: torch.Tensor, out: torch.Tensor,
                   w2: torch.Tensor, router: torch.Tensor, bias: torch.Tensor, logits: torch.Tensor, h2: torch.Tensor,
                   ticket: torch.Tensor, r: Routing, pdl: bool = False) -> None:
    """out = W RMSNorm(x; w1) in fp32 and, in the same launch, h2 = RMSNorm(x; w2) in fp32, its router logits and the
    choice of experts. ``ticket``: one int32 word, zero."""
    _twin_in_checks(x, w1, w, out)
    assert router.dtype == torch.bfloat16 and router.is_contiguous() and bias.numel() == router.shape[0]
    assert h2.shape == x.shape and h2.dtype == torch.float32 and h2.is_contiguous() and logits.is_contiguous()
    for lo, hi in _row_chunks(*x.shape):
        rc = _lib.cuda().rmlx_twin_in_router(
            x[lo:].data_ptr(), w1.data_ptr(), w2.data_ptr(), eps, width, x.shape[1], w.data_ptr(), w.shape[0], out[lo:].data_ptr(),
            out.stride(0), router.data_ptr(), bias.data_ptr(), router.shape[0], logits[lo:].data_ptr(), h2[lo:].data_ptr(),
            r.idx[lo:].data_ptr(), r.weights[lo:].data_ptr(), r.idx.shape[1], ticket.data_ptr(), hi - lo, int(pdl),
            _lib.stream_ptr())
        _lib.check(rc, "twin_in_router")
