"""Routing by corrected scores with identity experts, by biased logits with the softmax over the chosen
experts, or by sigmoids among the best groups beside experts that every token uses (csrc/kernels/moe_route.cu), and the grouped expert
feed-forward around it for any number of tokens: route -> rows sorted by expert -> gate/up with the gated
activation -> down. The combination with the output norm is ``combine_post_norm`` (postnorm_rows.cu)."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import _lib
from .parallel_block import _f32
from .post_norm import Pending, _chunks, gated_act, max_rows
from .quantized import xgemm
from .weights import LinearWeight

ROUTE_MAX_OUTPUTS, ROUTE_MAX_TOP = 512, 32       # of the routing kernel

_lib.register_cuda_sigs({
    "rmlx_route_max_outputs": ("", "i"),
    "rmlx_route_max_top": ("", "i"),
    "rmlx_route_corrected": ("pippppppiiiiip", "i"),
    "rmlx_route_chosen": ("pippppp" "iiiip", "i"),
    "rmlx_route_grouped": ("pipppp" "iiiiiifip", "i"),
    "rmlx_grouped_router": ("ppipppp" "iiiiiifip", "i"),
    "rmlx_route_scatter": ("pipppp" "iiiiiip", "i"),
    "rmlx_moe_combine_post_norm": ("pipppipfppiiiiip", "i"),
    "rmlx_postnorm_router": ("ppppfpii" "pppppp" "iiiiip", "i"),
    "rmlx_postnorm_expert": ("ppippiiiiifip", "i"),
    "rmlx_expert_out": ("piipippppp" "iiiiiip", "i"),
    "rmlx_sgemm_grouped": ("pipipipiiiiip", "i"),
})


@dataclass
class Routing:
    """Device arrays of one routed batch (views of preallocated buffers)."""
    idx: torch.Tensor            # int32 [T, top]; identity experts have idx >= experts
    weights: torch.Tensor        # fp32 [T, top]
    identity: Optional[torch.Tensor]   # fp32 [T] summed weight of the identity experts (None: there are none)
    counts: torch.Tensor         # int32 [experts]
    offsets: torch.Tensor        # int32 [experts + 1]
    row_of_pair: torch.Tensor    # int32 [T, top]; -1: no row


def route_corrected(logits: torch.Tensor, correction: torch.Tensor, experts: int, r: Routing, grouped: bool = True,
                    pdl: bool = False) -> None:
    """Chooses by softmax + correction, weights by the softmax alone. ``grouped``: also the experts' row ranges."""
    _lib.require_cuda_tensor(logits, correction, r.idx)
    t, outputs = logits.shape
    assert logits.dtype == correction.dtype == torch.float32 and correction.numel() == outputs
    rc = _lib.cuda().rmlx_route_corrected(
        logits.data_ptr(), logits.stride(0), correction.data_ptr(), r.idx.data_ptr(), r.weights.data_ptr(),
        r.identity.data_ptr(), r.counts.data_ptr() if grouped else None, r.offsets.data_ptr() if grouped else None, t,
        experts, outputs, r.idx.shape[1], int(pdl), _lib.stream_ptr())
    _lib.check(rc, "route_corrected")


def route_chosen(logits: torch.Tensor, bias: torch.Tensor, r: Routing, grouped: bool = True, pdl: bool = False) -> None:
    """Chooses by logits + bias, weights by the softmax over the chosen experts' alone (no identity experts)."""
    _lib.require_cuda_tensor(logits, bias, r.idx)
    t, experts = logits.shape
    assert logits.dtype == bias.dtype == torch.float32 and bias.numel() == experts
    rc = _lib.cuda().rmlx_route_chosen(
        logits.data_ptr(), logits.stride(0), bias.data_ptr(), r.idx.data_ptr(), r.weights.data_ptr(),
        r.counts.data_ptr() if grouped else None, r.offsets.data_ptr() if grouped else None, t, experts, r.idx.shape[1],
        int(pdl), _lib.stream_ptr())
    _lib.check(rc, "route_chosen")


@dataclass
class RouteGroups:
    """Groups of neighbouring experts of which a token may use the ``keep`` best; the weights' factor; how many experts
    behind the routed ones every token uses, with weight one."""
    count: int = 1
    keep: int = 1
    scale: float = 1.0
    always: int = 0


def route_grouped(logits: torch.Tensor, g: RouteGroups, r: Routing, grouped: bool = True, pdl: bool = False) -> None:
    """Chooses by sigmoid(logits) within the groups whose two largest have the largest sums; weights: the sigmoids times
    ``g.scale``. ``r`` has room for the chosen and the ``g.always`` experts."""
    _lib.require_cuda_tensor(logits, r.idx)
    t, experts = logits.shape
    assert logits.dtype == torch.float32 and r.counts.numel() == experts + g.always
    rc = _lib.cuda().rmlx_route_grouped(
        logits.data_ptr(), logits.stride(0), r.idx.data_ptr(), r.weights.data_ptr(), r.counts.data_ptr() if grouped else None,
        r.offsets.data_ptr() if grouped else None, t, experts, r.idx.shape[1] - g.always, g.count, g.keep, g.always, g.scale,
        int(pdl), _lib.stream_ptr())
    _lib.check(rc, "route_grouped")


def route_scatter(h: torch.Tensor, r: Routing, xs: torch.Tensor, always: int = 0, pdl: bool = False) -> None:
    """Copies every routed (token, slot) row of ``h`` into ``xs`` [T * top, width], sorted by expert. ``always``: how many
    of the experts (the last ones) have every token's row."""
    _lib.require_cuda_tensor(h, xs)
    t, top = r.idx.shape
    assert h.is_contiguous() and xs.is_contiguous() and xs.shape == (t * top, h.shape[1]) and xs.dtype == h.dtype
    rc = _lib.cuda().rmlx_route_scatter(h.data_ptr(), h.stride(0), r.idx.data_ptr(), r.counts.data_ptr(), xs.data_ptr(),
                                        r.row_of_pair.data_ptr(), t, top, r.counts.numel(), always, _f32(h), int(pdl),
                                        _lib.stream_ptr())
    _lib.check(rc, "route_scatter")


def _sgemm_grouped(x, w, offsets, out, max_rows, pdl):
    rc = _lib.cuda().rmlx_sgemm_grouped(x.data_ptr(), x.stride(0), w.data_ptr(), w.stride(1), offsets.data_ptr(),
                                        w.shape[0], out.data_ptr(), out.stride(0), max_rows, w.shape[1], w.shape[2],
                                        int(pdl), _lib.stream_ptr())
    _lib.check(rc, "sgemm_grouped")


def grouped_gated_ffn(xs: torch.Tensor, offsets: torch.Tensor, gate_up: LinearWeight, down: LinearWeight, limit: float,
                      tokens: int, scratch, act: torch.Tensor, y: torch.Tensor, pdl: bool = False) -> None:
    """y rows = expert feed-forward of the expert-sorted rows ``xs``; ``tokens`` bounds the rows of one expert.
    fp32 goes through ``scratch`` [rows, 2 n]."""
    if not _f32(xs):
        xgemm(xs, gate_up, offsets=offsets, out=act, swiglu=True, gate_limit=limit, pdl=pdl)
        xgemm(act, down, offsets=offsets, out=y, pdl=pdl)
        return
    _sgemm_grouped(xs, gate_up.w, offsets, scratch, tokens, pdl)
    gated_act(scratch, act, limit, pdl=pdl)
    _sgemm_grouped(act, down.w, offsets, y, tokens, pdl)


def combine_post_norm(y: torch.Tensor, r: Routing, w: torch.Tensor, eps: float, width: int, x: torch.Tensor,
                      h: torch.Tensor, pdl: bool = False) -> None:
    """x += RMSNorm(sum of weighted expert rows + identity weight * x) * w; h = x in the compute type."""
    _lib.require_cuda_tensor(y, w, x, h)
    t, ldx = x.shape
    assert x.dtype == torch.float32 and x.is_contiguous() and h.shape == x.shape and h.dtype == y.dtype
    rc = _lib.cuda().rmlx_moe_combine_post_norm(
        y.data_ptr(), y.stride(0), r.row_of_pair.data_ptr(), r.weights.data_ptr(), r.identity.data_ptr(),
        r.idx.shape[1], w.data_ptr(), eps, x.data_ptr(), h.data_ptr(), t, width, ldx, _f32(y), int(pdl),
        _lib.stream_ptr())
    _lib.check(rc, "moe_combine_post_norm")


# ------------------------------------------------------------------ decode (csrc/kernels/postnorm_gemv.cu)
def postnorm_router(x: torch.Tensor, pending: Pending, eps: float, width: int, x_out: torch.Tensor, w: torch.Tensor,
                    correction: torch.Tensor, experts: int, logits: torch.Tensor, ticket: torch.Tensor, r: Routing,
                    pdl: bool = False) -> None:
    """x_out = x + RMSNorm(pending), router logits and the choice. ``ticket``: one int32 word, zero."""
    _lib.require_cuda_tensor(x, x_out, w, logits, ticket)
    b, k = x.shape
    outputs, top = w.shape[0], r.idx.shape[1]
    assert w.dtype == torch.bfloat16 and w.is_contiguous() and logits.is_contiguous() and correction.numel() == outputs
    for lo, hi in _chunks(b, k):
        y = None if pending.y is None else pending.y[lo:].data_ptr()
        rc = _lib.cuda().rmlx_postnorm_router(
            w.data_ptr(), x[lo:].data_ptr(), y, _lib.ptr(pending.w), eps, x_out[lo:].data_ptr(), width, k,
            correction.data_ptr(), logits[lo:].data_ptr(), r.idx[lo:].data_ptr(), r.weights[lo:].data_ptr(),
            r.identity[lo:].data_ptr(), ticket.data_ptr(), hi - lo, experts, outputs, top, int(pdl), _lib.stream_ptr())
        _lib.check(rc, "postnorm_router")


def grouped_router(h: torch.Tensor, w: torch.Tensor, g: RouteGroups, logits: torch.Tensor, ticket: torch.Tensor, r: Routing,
                   pdl: bool = False) -> None:
    """Router logits of finished rows (fp32) and ``route_grouped``'s choice. ``ticket``: one int32 word, zero."""
    _lib.require_cuda_tensor(h, w, logits, ticket)
    b, k = h.shape
    assert h.dtype == torch.float32 and h.is_contiguous() and w.dtype == torch.bfloat16 and w.is_contiguous() and w.shape[1] == k
    assert logits.is_contiguous()
    for lo, hi in _chunks(b, k):
        rc = _lib.cuda().rmlx_grouped_router(
            w.data_ptr(), h[lo:].data_ptr(), k, logits[lo:].data_ptr(), r.idx[lo:].data_ptr(), r.weights[lo:].data_ptr(),
            ticket.data_ptr(), hi - lo, w.shape[0], r.idx.shape[1] - g.always, g.count, g.keep, g.always, g.scale, int(pdl),
            _lib.stream_ptr())
        _lib.check(rc, "grouped_router")


def postnorm_expert(x: torch.Tensor, w: torch.Tensor, limit: float, r: Routing, act: torch.Tensor, pdl: bool = False) -> None:
    """act [B * top, n] = gated activation of the chosen experts' [gate; up] projections of x (fp32)."""
    _lib.require_cuda_tensor(x, w, act)
    e, n2, k = w.shape
    assert x.shape[1] == k and w.is_contiguous() and act.shape == (r.idx.numel(), n2 // 2) and act.is_contiguous()
    rc = _lib.cuda().rmlx_postnorm_expert(w.data_ptr(), x.data_ptr(), k, r.idx.data_ptr(), act.data_ptr(), act.stride(0),
                                          x.shape[0], r.idx.shape[1], n2 // 2, e, limit, int(pdl), _lib.stream_ptr())
    _lib.check(rc, "postnorm_expert")


def expert_out(act: torch.Tensor, w: torch.Tensor, r: Routing, x: torch.Tensor, y: torch.Tensor, pdl: bool = False) -> None:
    """y = sum of the slots' weighted down projections + identity weight * x (without identity weights: the sum alone)."""
    _lib.require_cuda_tensor(act, w, x, y)
    e, rows, k = w.shape
    b, ldx = x.shape
    assert y.shape == x.shape and act.stride(0) >= k and w.is_contiguous()
    rc = _lib.cuda().rmlx_expert_out(w.data_ptr(), rows, k, act.data_ptr(), act.stride(0), r.idx.data_ptr(),
                                     r.weights.data_ptr(), _lib.ptr(r.identity), x.data_ptr(), y.data_ptr(), ldx, b, ldx,
                                     r.idx.shape[1], e, int(pdl), _lib.stream_ptr())
    _lib.check(rc, "expert_out")


def expert_decode_fits(k: int, top: int) -> bool:
    """Whether ``expert_out`` can stage ``top`` activations of ``k`` values."""
    return max_rows(k * top) > 0
