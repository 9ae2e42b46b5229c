"""Nizorax on the GPU against the plain restatement in ``oracle/nizorax.py``: every mechanism alone, then the model through
its ragged batches, its decode engine, the serving engine and the command line, in 32-bit (tight) and bf16."""
import io
import json
import struct
import sys
from dataclasses import replace

import pytest
import torch
from oracle import nizorax as O
from torch.nn.functional import pad as fpad

from rmlx_b200.config import (DifferentialAttentionSpec, GroupedFfSpec, LightningSpec, LoopSpec, NizoraxConfig, PolyNormFfSpec,
                              RotarySpec, SamplerConfig, SandwichLayerSpec, SchedulerConfig)
from rmlx_b200.models import nizorax as M
from rmlx_b200.models.ragged import Entry, RaggedBatch, query_tiles
from rmlx_b200.models.ragged_model import Buffers, StepContext
from rmlx_b200.models.sandwich_decode import SandwichDecode
from rmlx_b200.ops import parallel_block as P
from rmlx_b200.ops import routed as R
from rmlx_b200.ops import sandwich as W
from rmlx_b200.ops import scan as S
from rmlx_b200.ops import twin_norm as TN
from rmlx_b200.serve.engine import ServingEngine

pytestmark = pytest.mark.gpu
BF, F32, D = torch.bfloat16, torch.float32, torch.float64
pad8 = P.pad8
LLAMA = {"factor": 5.0, "original": 64.0, "high": 4.0, "low": 0.7}


def rel(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    return float((got - want).norm() / want.norm().clamp_min(1e-30))


def worst_row(got, want):
    """Largest error of a row of logits (mean taken off) over the rms of the logits."""
    d = got.double().cpu() - want.double().cpu()
    d = d - d.mean(-1, keepdim=True)
    return float(d.pow(2).mean(-1).sqrt().max() / want.double().pow(2).mean().sqrt())


def rand(seed):
    g = torch.Generator().manual_seed(seed)
    return lambda *s: torch.randn(*s, generator=g)


def i32(x, dev):
    return torch.tensor(x, dtype=torch.int32, device=dev)


def shuffled_pages(lens, seed=5):
    """Block table [sequences, pages] of pages in shuffled order (page 0 stays reserved), and their count."""
    npg = [(n + 15) // 16 for n in lens]
    order = torch.randperm(sum(npg), generator=torch.Generator().manual_seed(seed)) + 1
    table, at = torch.zeros(len(lens), max(npg), dtype=torch.int32), 0
    for i, n in enumerate(npg):
        table[i, :n] = order[at:at + n].int()
        at += n
    return table, sum(npg) + 1


# ------------------------------------------------------------------ differential attention
class TwoMaps:
    """q, k (two maps each) and v of several sequences in pages; the maps' difference by the oracle."""

    def __init__(self, dev, lens, hq, hkv, dk, dv, dtype=BF, seed=0, lam=0.6, diff=0.25, eps=1e-4, sharp=1.0):
        r = rand(seed)
        self.dev, self.lens, self.hq, self.hkv, self.dk, self.dv, self.dtype = dev, lens, hq, hkv, dk, dv, dtype
        self.q, self.k = [r(n, hq, 2, dk).to(dtype) for n in lens], [r(n, hkv, 2, dk).to(dtype) for n in lens]
        self.v, self.scale = [r(n, hkv, dv).to(dtype) for n in lens], sharp * dk ** -0.5
        self.lam, self.diff, self.eps = lam, diff, eps
        self.mods, self.pair = P.ScoreMods(self.scale), P.MapDiff(lam, 1.0 - diff, eps)

    def build(self):
        table, count = shuffled_pages(self.lens)
        kc = torch.zeros(count, self.hkv, 16, 2, pad8(self.dk), dtype=self.dtype)
        vc = torch.zeros(count, self.hkv, 16, pad8(self.dv), dtype=self.dtype)
        for s, n in enumerate(self.lens):
            for t in range(n):
                kc[table[s, t // 16], :, t % 16, :, :self.dk] = self.k[s][t]
                vc[table[s, t // 16], :, t % 16, :self.dv] = self.v[s][t]
        return kc.flatten(3).to(self.dev), vc.to(self.dev), table.to(self.dev)

    def want(self, rows, window):
        outs = {}
        for s in {s for s, _ in rows}:
            q, k = (x[s].double().permute(1, 2, 0, 3) for x in (self.q, self.k))
            outs[s] = O.two_maps(q, k, self.v[s].double().permute(1, 0, 2), O.visible(self.lens[s], window or None), self.scale,
                                 self.lam, self.diff, self.eps)
        return torch.stack([outs[s][:, t] for s, t in rows])

    def every_kernel(self, rows, starts, window):
        """The rows (sequences' tails from ``starts``) through every attention kernel that takes them."""
        kc, vc, table = self.build()
        q = torch.zeros(len(rows), self.hq, 2, pad8(self.dk), dtype=self.dtype)
        for i, (s, t) in enumerate(rows):
            q[i, ..., :self.dk] = self.q[s][t]
        q = q.to(self.dev)
        pos, seq = i32([t for _, t in rows], self.dev), i32([s for s, _ in rows], self.dev)
        new = lambda: torch.full((len(rows), self.hq, pad8(self.dv)), 5.0, dtype=self.dtype, device=self.dev)   # noqa: E731
        outs = {"any": P.attention_any(q, kc, vc, table, pos, seq, self.mods, new(), window=window, diff=self.pair, vdim=self.dv)}
        if self.dtype == BF and P.prefill_scored_supported(pad8(self.dk), pad8(self.dv)):
            lens = [n - lo for n, lo in zip(self.lens, starts)]
            firsts = [sum(lens[:i]) for i in range(len(lens))]
            tiles = query_tiles(firsts, lens, starts, list(range(len(lens))), 128)
            outs["prompt"] = P.flash_prefill_diff(q, kc, vc, table, i32(tiles, self.dev), self.scale, self.pair, self.dv, new(),
                                                  window=window)
            for splits in (1, 3):
                scr = P.ScoredDecodeScratch(len(rows), 2 * self.hq, self.hkv, pad8(self.dv), splits, self.dev)
                outs[f"decode{splits}"] = P.flash_decode_scored(kc, vc, table, pos, self.mods, new(), scr, self.hq, self.dk, self.dv,
                                                                q=q, table_rows=seq, window=window, diff=self.pair)
        for n, o in outs.items():
            assert not o[..., self.dv:].any(), n
        return {n: o[..., :self.dv] for n, o in outs.items()}


SHAPES = [(4, 2, 32, 40), (3, 3, 20, 72), (8, 1, 128, 128), (12, 1, 64, 104), (40, 2, 16, 64), (2, 1, 136, 24), (2, 2, 24, 200)]


@pytest.mark.parametrize("shape", SHAPES, ids=str)
@pytest.mark.parametrize("dtype,tol", [(F32, 5e-6), (BF, 1.2e-2)])
@pytest.mark.parametrize("window", [0, 1, 16, 37, 130, 1000])
def test_differential_attention(dev, shape, dtype, tol, window):
    h = TwoMaps(dev, [3, 18, 300], *shape, dtype=dtype)
    starts = [0, 1, 45]
    rows = [(s, t) for s, lo in enumerate(starts) for t in range(lo, h.lens[s])]
    want = h.want(rows, window)
    for name, got in h.every_kernel(rows, starts, window).items():
        assert rel(got, want) < tol, name


def test_window_edges_stand_out(dev):
    """The first key a window holds carries most of one query's weight in one of the maps; the key before it, as strong,
    none. Another window would be far off."""
    for window in (15, 16, 17, 64, 100):
        for m in (0, 1):
            h = TwoMaps(dev, [260], 2, 1, 64, 32, seed=7)
            picks = [110, 150, 191, 255]
            for t in picks:
                for key in (t - window + 1, t - window):
                    h.k[0][key, :, m] = (h.q[0][t, 0, m].float() * 3).to(BF)
            rows = [(0, t) for t in range(100, 260)]
            want, at = h.want(rows, window), [t - 100 for t in picks]
            assert rel(h.want(rows, window + 1)[at], want[at]) > 0.2 and rel(h.want(rows, window - 1)[at], want[at]) > 0.2
            for name, got in h.every_kernel(rows, [100], window).items():
                assert rel(got, want) < 1.5e-2, (name, window)
                for t in at:
                    assert rel(got[t], want[t]) < 3e-2, (name, window, t)


@pytest.mark.parametrize("m", [0, 1])
def test_a_far_key_among_hundreds(dev, m):
    """One key at a page border far away takes one map over."""
    h = TwoMaps(dev, [700], 3, 1, 40, 48, seed=3)
    for t, key in ((699, 16), (650, 15), (600, 0), (512, 255)):
        h.k[0][key, :, m] = (h.q[0][t, 1, m].float() * 4).to(BF)
    rows = [(0, t) for t in range(500, 700)]
    want = h.want(rows, 0)
    lost = TwoMaps(dev, [700], 3, 1, 40, 48, seed=3).want(rows, 0)
    assert rel(lost[[199, 150, 100, 12]], want[[199, 150, 100, 12]]) > 0.3
    for name, got in h.every_kernel(rows, [500], 0).items():
        for t in (199, 150, 100, 12):
            assert rel(got[t], want[t]) < 3e-2, (name, t)


def turned(raw, spec, pos):
    """Rows [heads, 2, dim] after rotation at ``pos``, by the oracle (rows of a longer sequence)."""
    x = torch.zeros(*raw.shape[:2], pos + 1, raw.shape[-1], dtype=D)
    x[:, :, pos] = raw
    return O.rotate_neighbours(x, spec)[:, :, pos]


ROTARY = [{"base": 500.0, "dims": 20}, {"base": 1e4, "dims": 24, "scaling": LLAMA}, {"base": 1e4, "dims": 0},
          {"base": 7e4, "dims": 6, "scaling": {"factor": 1.5, "original": 8.0, "high": 2.0, "low": 1.9}}]
ROT_ID = lambda r: f"{r['dims']}{'s' if 'scaling' in r else ''}"          # noqa: E731


@pytest.mark.parametrize("dtype,tol", [(F32, 2e-6), (BF, 5e-3)])
@pytest.mark.parametrize("hq,hkv,dk,dv", [(3, 1, 24, 10), (6, 3, 72, 40), (2, 2, 300, 8), (5, 5, 27, 33)])
@pytest.mark.parametrize("rot", ROTARY, ids=ROT_ID)
def test_rotation_of_both_maps_and_append(dev, dtype, tol, hq, hkv, dk, dv, rot):
    r = rand(1)
    nq, nk, nv = hq * 2 * dk, hkv * 2 * dk, hkv * dv
    pos, seq = list(range(14, 31)) + list(range(20)) + [90], [0] * 17 + [1] * 20 + [2]
    t = len(pos)
    raw = r(t, pad8(nq + nk + nv)).to(dtype)
    f = TN.rotary_frequencies(rot["base"], rot["dims"], rot.get("scaling"))[0]
    kc = torch.zeros(12, hkv, 16, 2 * pad8(dk), dtype=dtype, device=dev)
    vc = torch.zeros(12, hkv, 16, pad8(dv), dtype=dtype, device=dev)
    table = i32([[4, 2, 8, 0, 0, 0], [7, 1, 3, 0, 0, 0], [0, 0, 0, 0, 0, 9]], dev)
    q = torch.full((t, hq, 2, pad8(dk)), 5.0, dtype=dtype, device=dev)
    TN.rotary_norm_append(raw.to(dev), None, f.float().to(dev), 1.0, 0.0, q, kc, vc, table, i32(pos, dev), i32(seq, dev), hq, dk, dv,
                          neighbours=True, norm=False, maps=2)
    d, keys = raw.double(), kc.view(12, hkv, 16, 2, pad8(dk))
    for i in (0, 3, 16, 17, 36, t - 1):
        assert rel(q[i, ..., :dk], turned(d[i, :nq].view(hq, 2, dk), rot, pos[i])) < tol
        page, off = int(table[seq[i], pos[i] // 16]), pos[i] % 16
        assert rel(keys[page, :, off, :, :dk], turned(d[i, nq:nq + nk].view(hkv, 2, dk), rot, pos[i])) < tol
        assert rel(vc[page, :, off, :dv], d[i, nq + nk:nq + nk + nv].view(hkv, dv)) < tol
    assert not q[..., dk:].any() and not keys[..., dk:].any() and not vc[..., dv:].any() and not kc[[0, 5, 6, 10]].any()


def test_rotation_of_neighbours_with_a_norm_and_one_map(dev):
    """The append kernel's parts in other combinations: neighbours with bias, factor and norm, one map."""
    r, hq, hkv, dk, dv, rot = rand(4), 4, 2, 40, 24, ROTARY[0]
    raw, bias = r(3, pad8(hq * dk + hkv * (dk + dv))), 0.3 * r(hq * dk + hkv * (dk + dv))
    f = TN.rotary_frequencies(rot["base"], rot["dims"])[0].float().to(dev)
    kc, vc = torch.zeros(4, hkv, 16, dk, device=dev), torch.zeros(4, hkv, 16, dv, device=dev)
    q = torch.empty(3, hq, dk, device=dev)
    TN.rotary_norm_append(raw.to(dev), bias.to(dev), f, 1.3, 1e-3, q, kc, vc, i32([[1], [2], [3]], dev), i32([5, 0, 15], dev), None,
                          hq, dk, dv, neighbours=True)
    d = raw.double()[:, :len(bias)] + bias.double()
    for i, pos in enumerate((5, 0, 15)):
        both = turned(d[i, :(hq + hkv) * dk].view(-1, 1, dk), rot, pos)[:, 0]
        both[:, :rot["dims"]] *= 1.3
        want = O.rms_norm(both, 1e-3)
        assert rel(q[i], want[:hq]) < 2e-6 and rel(kc[i + 1, :, pos], want[hq:]) < 2e-6


@pytest.mark.parametrize("shape", [(4, 2, 32, 40), (2, 2, 20, 72), (40, 2, 64, 64), (9, 1, 128, 128), (3, 1, 27, 30)], ids=str)
@pytest.mark.parametrize("window,rot", [(0, ROTARY[0]), (17, {"base": 1e4, "dims": 18, "scaling": LLAMA}), (64, ROTARY[2])])
def test_fused_rotation_append_attention(dev, shape, window, rot):
    """The decode form: one launch on the projection's fp32 rows."""
    hq, hkv, dk, dv = shape
    r, lens = rand(3), [1, 16, 17, 200]
    h = TwoMaps(dev, lens, *shape, seed=2)
    nq, nk, nv = hq * 2 * dk, hkv * 2 * dk, hkv * dv
    raw = r(4, nq + nk + nv + 5)
    d = raw.double()
    for s, n in enumerate(lens):                          # the oracle's view of the new token
        h.q[s][n - 1] = turned(d[s, :nq].view(hq, 2, dk), rot, n - 1).to(BF)
        h.k[s][n - 1] = turned(d[s, nq:nq + nk].view(hkv, 2, dk), rot, n - 1).to(BF)
        h.v[s][n - 1] = d[s, nq + nk:nq + nk + nv].view(hkv, dv).to(BF)
    want_k, want_v, table = h.build()
    kc, vc = want_k.clone(), want_v.clone()
    for s, n in enumerate(lens):                          # the slot of the new token starts dirty
        kc.view(*kc.shape[:3], 2, -1)[table[s, (n - 1) // 16], :, (n - 1) % 16, :, :dk] = 9.0
        vc[table[s, (n - 1) // 16], :, (n - 1) % 16, :dv] = -9.0
    f = TN.rotary_frequencies(rot["base"], rot["dims"], rot.get("scaling"))[0]
    for splits in (1, 5):
        out = torch.zeros(4, hq, pad8(dv), dtype=BF, device=dev)
        scr = P.ScoredDecodeScratch(4, 2 * hq, hkv, pad8(dv), splits, dev)
        P.flash_decode_scored(kc, vc, table, i32([n - 1 for n in lens], dev), h.mods, out, scr, hq, dk, dv, raw=raw.to(dev),
                              window=window, head_norm=True, normed=False, inv_freq=f.float().to(dev), neighbours=True, diff=h.pair)
        assert rel(out[..., :dv], h.want([(s, n - 1) for s, n in enumerate(lens)], window)) < 1.2e-2
        assert rel(kc, want_k) < 3e-3 and rel(vc, want_v) < 3e-3


# ------------------------------------------------------------------ rows: norms, convolution, activation
def padded(x, dev, dtype=F32):
    return fpad(x, (0, pad8(x.shape[-1]) - x.shape[-1])).to(dev, dtype)


def affine(r, width, dev):
    """(weight, bias) and the kernels' [2, padded] tensor."""
    w, b = 1 + 0.3 * r(width), 0.4 * r(width)
    return (w.double(), b.double()), padded(torch.stack([w, b]), dev)


def routing_of(order, weights, dev):
    """Expert rows anywhere in a buffer: (token, slot) -> row."""
    t, top = order.shape
    i = lambda *s: torch.zeros(*s, dtype=torch.int32, device=dev)         # noqa: E731
    return R.Routing(i(t, top), weights.to(dev), None, i(1), i(2), order.to(dev))


@pytest.mark.parametrize("width", [1, 20, 104, 1030, 2100, 4096, 9000])
@pytest.mark.parametrize("t", [1, 7])
@pytest.mark.parametrize("dtype,tol", [(F32, 3e-6), (BF, 4e-3)])
def test_output_norm_residual_and_norm(dev, width, t, dtype, tol):
    r, eps = rand(width), 1e-2
    x0, y = 3 * r(t, width) + 2, (2 * r(t, width) - 5).to(dtype)          # means far from zero
    (wy, by), pa = affine(r, width, dev)
    (wh, bh), ph = affine(r, width, dev)
    x = padded(x0, dev)
    h = torch.full_like(x, 9.0, dtype=dtype)
    W.sandwich_norm(x, None, None, ph, h, eps, width)
    assert rel(h[:, :width], O.layer_norm(x0.double(), eps, wh, bh)) < tol and not h[:, width:].any() and torch.equal(x, padded(x0, dev))
    want = x0.double() + O.layer_norm(y.double(), eps, wy, by)
    W.sandwich_norm(x, padded(y, dev, dtype), pa, ph, h, eps, width)
    assert rel(x[:, :width], want) < 2e-6 and not x[:, width:].any()
    assert rel(h[:, :width], O.layer_norm(want, eps, wh, bh)) < tol and not h[:, width:].any()
    x2 = padded(x0, dev)
    W.sandwich_norm(x2, padded(y, dev, dtype), pa, None, None, eps, width)
    assert torch.equal(x, x2)
    for top in (1, 3, 6):                                 # experts' rows: slots in any order, more than four of them
        ye = torch.zeros(t * top, pad8(width) + 8)
        ye[:, :width] = r(t * top, width)
        order = torch.randperm(t * top, generator=torch.Generator().manual_seed(top)).int().view(t, top)
        wt = torch.rand(t, top, generator=torch.Generator().manual_seed(top))
        yd = ye.to(dtype)
        total = (wt.double()[:, :, None] * yd[:, :width].double()[order.long()]).sum(1)
        want = x0.double() + O.layer_norm(total, eps, wy, by)
        x = padded(x0, dev)
        W.sandwich_norm(x, yd.to(dev), pa, ph, h, eps, width, routing=routing_of(order, wt, dev))
        assert rel(x[:, :width], want) < 3e-6 and rel(h[:, :width], O.layer_norm(want, eps, wh, bh)) < tol


def test_many_rows_share_blocks(dev):
    """Enough rows for the form with two rows a block, an odd number of them."""
    t, width, r = 2401, 300, rand(1)
    x0, y = r(t, width), r(t, width).to(BF)
    (wy, by), pa = affine(r, width, dev)
    (wh, bh), ph = affine(r, width, dev)
    x = padded(x0, dev)
    h = torch.full_like(x, 9.0, dtype=BF)
    W.sandwich_norm(x, padded(y, dev, BF), pa, ph, h, 1e-5, width)
    want = x0.double() + O.layer_norm(y.double(), 1e-5, wy, by)
    assert rel(x[:, :width], want) < 2e-6 and rel(h[:, :width], O.layer_norm(want, 1e-5, wh, bh)) < 4e-3
    assert rel(x[-1, :width], want[-1]) < 2e-6


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7])
@pytest.mark.parametrize("dtype,tol", [(F32, 1e-6), (BF, 4e-3)])
def test_short_convolution_in_portions(dev, taps, dtype, tol):
    """Three sequences cut differently, portions shorter than the window, single rows; other slots stay as they are."""
    width, lens, r = 52, [30, 41, 9], rand(taps)
    w = r(width, taps)
    hs = [r(n, width).to(dtype) for n in lens]
    want = [O.short_conv(h.double(), w.double()) for h in hs]
    if taps > 1:                                          # on the CPU: one token off is far off
        assert rel(O.short_conv(hs[0].double(), torch.roll(w, 1, 1).double()), want[0]) > 0.3
    wd = padded(w.t().contiguous(), dev)
    pool = torch.full((5, (taps - 1) * pad8(width) + 4), 3.0, device=dev)
    carried = None if taps == 1 else pool[:, :(taps - 1) * pad8(width)].unflatten(1, (taps - 1, pad8(width)))
    slots = [3, 0, 2]
    if taps > 1:
        carried[slots] = 0.0
    at, got = [0, 0, 0], [[], [], []]
    for cut in ([2, 1, 0], [1, 19, 3], [0, 2, 1], [17, 1, 0], [1, 1, 1], [9, 17, 4]):
        live = [i for i in range(3) if cut[i]]
        rows = torch.cat([hs[i][at[i]:at[i] + cut[i]] for i in live])
        runs, lo = [], 0
        for i in live:
            runs.append([lo, cut[i], slots[i], at[i]])
            lo += cut[i]
        out = torch.full((lo, pad8(width)), 8.0, dtype=dtype, device=dev)
        W.short_conv(padded(rows, dev, dtype), wd, carried, out, i32([slots[i] for i in live for _ in range(cut[i])], dev),
                     runs=i32(runs, dev))
        for i, (a, n, _, _) in zip(live, runs):
            got[i].append(out[a:a + n, :width].cpu())
            at[i] += n
    assert at == lens
    for g, v in zip(got, want):
        assert rel(torch.cat(g), v) < tol
    assert (pool[[1, 4]] == 3.0).all() and (pool[:, (taps - 1) * pad8(width):] == 3.0).all()
    # every row a sequence of its own
    if taps > 1:
        out = torch.empty(3, pad8(width), dtype=dtype, device=dev)
        nxt = [r(1, width).to(dtype) for _ in range(3)]
        W.short_conv(padded(torch.cat(nxt), dev, dtype), wd, carried, out, i32(slots, dev))
        for i in range(3):
            assert rel(out[i, :width], O.short_conv(torch.cat([hs[i], nxt[i]]).double(), w.double())[-1]) < tol


@pytest.mark.parametrize("width,taps", [(60, 3), (4096, 4), (300, 1), (5000, 2), (9000, 6)])
@pytest.mark.parametrize("dtype,tol", [(F32, 5e-6), (BF, 6e-3)])
def test_decode_rows_through_norms_and_convolution(dev, width, taps, dtype, tol):
    r, b, eps = rand(taps), 3, 1e-3
    (wy, by), pa = affine(r, width, dev)
    (wh, bh), ph = affine(r, width, dev)
    w = 0.5 * r(width, taps)
    wd = padded(w.t().contiguous(), dev)
    carried = torch.zeros(4, max(taps - 1, 1), pad8(width), device=dev) if taps > 1 else None
    slots, past = [2, 0, 3], [[], [], []]
    x0 = r(b, width)
    x, want = padded(x0, dev), x0.double()
    for step in range(5):
        y = (2 * r(b, width) + 1).to(dtype)
        h = torch.full((b, pad8(width)), 7.0, dtype=dtype, device=dev)
        W.sandwich_step(x, padded(y, dev, dtype), pa, ph, h, eps, width, (wd, carried, i32(slots, dev)))
        want = want + O.layer_norm(y.double(), eps, wy, by)
        assert rel(x[:, :width], want) < 3e-6 and not x[:, width:].any()
        n = O.layer_norm(want, eps, wh, bh)
        for i in range(b):
            past[i].append(n[i])
            assert rel(h[i, :width], O.short_conv(torch.stack(past[i]), w.double())[-1]) < tol, step
    before = x.clone()
    W.sandwich_step(x, None, None, ph, h, eps, width)     # no sublayer pending, no convolution
    assert torch.equal(x, before) and rel(h[:, :width], O.layer_norm(want, eps, wh, bh)) < tol
    ye = r(b * 3, width).to(dtype)
    order, wt = torch.randperm(b * 3, generator=torch.Generator().manual_seed(1)).int().view(b, 3), torch.rand(b, 3)
    W.sandwich_step(x, padded(ye, dev, dtype), pa, ph, h, eps, width, routing=routing_of(order, wt, dev))
    total = (wt.double()[:, :, None] * ye.double()[order.long()]).sum(1)
    assert rel(x[:, :width], want + O.layer_norm(total, eps, wy, by)) < 3e-6


@pytest.mark.parametrize("width", [5, 72, 1000, 5000, 21504, 25000])
@pytest.mark.parametrize("dtype,tol", [(F32, 3e-6), (BF, 5e-3)])
def test_polynomial_of_normed_powers(dev, width, dtype, tol):
    r, act = rand(width), torch.tensor([0.7, -0.4, 1.3, 0.25])
    z = (2 * r(5, width)).to(dtype)
    ld = (width + 63) // 64 * 64
    zd = fpad(z, (0, ld - width), value=4.0).to(dev)      # what lies past the width is nobody's
    out = torch.full_like(zd, 6.0)
    want = O.poly_norm(z.double(), 1e-2, act.double())
    W.poly_norm(zd, act.to(dev), 1e-2, width, out)
    assert rel(out[:, :width], want) < tol and not out[:, width:].any()
    W.poly_norm(zd, act.to(dev), 1e-2, width, zd)         # in place
    assert torch.equal(zd, out)


@pytest.mark.parametrize("b", [1, 3, 6])
@pytest.mark.parametrize("n,width", [(40, 72), (1030, 700), (300, 9000)])
def test_decode_projections(dev, b, n, width):
    """Activation and norm with gate in the staging of the projection that follows."""
    r, k = rand(b), (width + 63) // 64 * 64
    w = fpad((r(n, width) / width ** 0.5).to(BF), (0, k - width)).to(dev)
    wd, act = w[:, :width].double().cpu(), torch.tensor([0.9, 0.3, -0.6, 0.1])
    z, y = 2 * r(b, width), torch.full((b, n), 7.0, device=dev)
    W.poly_out(fpad(z, (0, k - width), value=5.0).to(dev), act.to(dev), 1e-3, width, w, y)
    assert rel(y, O.poly_norm(z.double(), 1e-3, act.double()) @ wd.T) < 5e-6
    gate, norm = 3 * r(b, width), 1 + 0.2 * r(width)
    wide = torch.full((b, 2 * k), 4.0)                    # o and gate side by side, strangers past the width
    wide[:, :width], wide[:, k:k + width] = z, gate
    wide = wide.to(dev)
    W.gated_out(wide[:, :k], wide[:, k:], norm.to(dev), 1e-3, w, y)
    want = O.rms_norm(z.double(), 1e-3, norm.double()) * torch.sigmoid(gate.double())
    assert rel(y, want @ wd.T) < 5e-6


# ------------------------------------------------------------------ lightning attention
LIGHT = [LightningSpec(3, 7, 12, [0.3, 0.9, 0.999]), LightningSpec(2, 16, 33, [1.0, 0.5]), LightningSpec(1, 64, 64, [0.97]),
         LightningSpec(2, 100, 20, [0.8, 0.99]), LightningSpec(1, 200, 264, [0.95]), LightningSpec(4, 128, 128, [0.6, 0.9, 0.99, 0.9995])]
LIGHT_ID = lambda m: f"{m.heads}-{m.dim}-{m.vdim}"                        # noqa: E731


def one_layer(mixer, mlp=None, width=40, taps=3, seed=0):
    """(config, checkpoint tensors in fp32) of a model of one layer."""
    cfg = NizoraxConfig(16, width, [SandwichLayerSpec(mixer, mlp)], 1e-5, taps=taps).validate()
    return cfg, {k: v.float() for k, v in M.random_tensors(cfg, seed).items()}


class MixerCase:
    """A model of one layer without feed-forward; its mixer over whole sequences by the oracle."""

    def __init__(self, dev, mixer, dtype, width=40):
        self.dev, self.dtype, self.width = dev, dtype, width
        self.cfg, t = one_layer(mixer, None, width)
        self.t = {k: v if v.dim() == 1 else v.to(dtype).float() for k, v in t.items()}
        self.model = M.NizoraxModel(M.build_weights(self.cfg, self.t, dev, dtype))
        self.mw, self.w = self.model.w.layers[0].mix, {k[7:]: v.double() for k, v in self.t.items() if k.startswith("l0.mix.")}
        self.cache = self.model.new_cache(80, max_seqs=6)

    def project(self, a):
        return (a.double() @ self.mw.w_o.w.double().T)[:, :self.width].cpu()

    def run(self, forward, hs, cuts):
        """The sequences' rows in portions (all that are left to cut share a batch), continued on the cache."""
        for i in range(len(hs)):
            self.cache.add_sequence(i)
        got, at = [[] for _ in hs], [0] * len(hs)
        for cut in cuts:
            live = [i for i in range(len(hs)) if cut[i]]
            for i in live:
                self.cache.reserve(i, cut[i])
            b = RaggedBatch.plan([Entry(i, [0] * cut[i]) for i in live], self.cache, 0).upload(self.dev)
            c = StepContext(b.num_tokens, Buffers(256, self.dev), self.cache, self.cache.block_table, b.positions, b.token_seq,
                            b.token_seq, b.runs, b)
            x = padded(torch.cat([hs[i][at[i]:at[i] + cut[i]] for i in live]), self.dev, self.dtype)
            out, lo = self.project(forward(0, self.mw, x, c)), 0
            for i in live:
                got[i].append(out[lo:lo + cut[i]])
                lo += cut[i]
                at[i] += cut[i]
                self.cache.commit(i, cut[i])
        assert at == [len(h) for h in hs]
        return [torch.cat(g) for g in got]


CUTS = ([1, 1, 2, 3], [0, 2, 17, 16], [0, 1, 1, 1], [0, 1, 30, 13], [0, 0, 130, 0])
LENS = [1, 5, 180, 33]


@pytest.mark.parametrize("spec", LIGHT, ids=LIGHT_ID)
@pytest.mark.parametrize("dtype,tol", [(F32, 5e-6), (BF, 1.5e-2)])
def test_lightning_attention_in_portions(dev, spec, dtype, tol):
    c = MixerCase(dev, spec, dtype)
    hs = [rand(40 + i)(n, c.width).to(dtype) for i, n in enumerate(LENS)]
    for g, h in zip(c.run(c.model.lightning, hs, CUTS), hs):
        assert rel(g, O.lightning(c.w, spec.to_json(), 1e-5, h.double())) < tol


@pytest.mark.parametrize("spec", [DifferentialAttentionSpec(4, 2, 28, 20, 0.3, RotarySpec(100.0, 12, LLAMA), 0.3, 9),
                                  DifferentialAttentionSpec(3, 1, 136, 12, 0.1, RotarySpec(1e4, 136), 0.7)], ids=["narrow", "wide"])
@pytest.mark.parametrize("dtype,tol", [(F32, 2e-5), (BF, 4e-2)])
def test_differential_attention_in_portions(dev, spec, dtype, tol):
    c = MixerCase(dev, spec, dtype)
    hs = [rand(40 + i)(n, c.width).to(dtype) for i, n in enumerate(LENS)]
    for g, h in zip(c.run(c.model.attention, hs, CUTS), hs):
        assert rel(g, O.differential_attention(c.w, spec.to_json(), 1e-5, h.double())) < tol


@pytest.mark.parametrize("dtype,tol", [(F32, 2e-5), (BF, 1e-2)])
def test_states_decay_exactly_over_a_long_past(dev, dtype, tol):
    """One strong key at the start is read back hundreds of tokens later through a slow decay: a lost or repeated decay
    step shows in 32-bit, a lost state in both."""
    h, n, d, t = 2, 24, 40, 600
    r = rand(9)
    q, k, v = 0.01 * r(t, h * n), 0.01 * r(t, h * n), r(t, h * d)
    k[3], q[t - 1] = 6.0, 3.0
    decay = torch.tensor([0.998, 0.9995])
    wide = torch.zeros(t, 2 * h * n + h * d, dtype=dtype, device=dev)     # one row stride for q, k and v
    wide.copy_(torch.cat([q, k, v], 1))
    back = wide.double().cpu()
    hf = lambda x: O.silu(O.heads_first(x, h))                            # noqa: E731
    parts = [hf(x) for x in torch.split(back, [h * n, h * n, h * d], 1)]
    want = O.heads_last(O.decayed_state(*parts, decay.double()))
    assert rel(O.heads_last(O.decayed_state(*parts, torch.tensor([0.9979, 0.9994], dtype=D)))[-1], want[-1]) > 1e-2
    state, o = torch.zeros(3, h, n, d, device=dev), torch.zeros(t, h * d, device=dev)
    qd, kd, vd = wide[:, :h * n], wide[:, h * n:2 * h * n], wide[:, 2 * h * n:]
    rec = torch.empty(t * h * S.record(n, d, True), device=dev)
    S.lightning_scan(qd, kd, vd, decay.to(dev), state, o, rec, runs=i32([[0, t, 1, 0]], dev))
    assert rel(o[-1], want[-1]) < tol and rel(o, want) < tol and not state[[0, 2]].any()


@pytest.mark.parametrize("spec", LIGHT + [LightningSpec(2, 250, 300, [0.9, 0.7])], ids=LIGHT_ID)
@pytest.mark.parametrize("b", [1, 3])
def test_lightning_decode_step(dev, spec, b):
    c = MixerCase(dev, spec, BF)
    state = c.cache.layer_state(0, "state")
    slots = torch.randperm(6, generator=torch.Generator().manual_seed(1))[:b].int().to(dev)
    h = rand(b)(b, 6, c.width)
    want = [O.lightning(c.w, spec.to_json(), 1e-5, x.double()) for x in h]
    _, at_k, at_v, at_g = c.mw.at
    o, y = torch.zeros(b, c.mw.w_o.k, device=dev), torch.zeros(b, pad8(c.width), device=dev)
    for t in range(6):
        raw = (padded(h[:, t], dev).double() @ c.mw.w_in.w.double().T).float()
        W.lightning_step(raw, at_k, at_v, c.mw.decay, slots, state, o)
        W.gated_out(o, raw[:, at_g:], c.mw.norm, 1e-5, c.mw.w_o.w, y)
        assert rel(y[:, :c.width], torch.stack([w[t] for w in want])) < 2e-5, t
    assert int((c.cache.state.abs().sum(1) > 0).sum()) == b               # other slots are untouched


@pytest.mark.parametrize("size", [20, 130, 512, 1500, 5000])
@pytest.mark.parametrize("dtype,tol", [(F32, 1e-6), (BF, 4e-3)])
def test_norm_with_a_sigmoid_gate(dev, size, dtype, tol):
    r = rand(size)
    o, z, w = r(9, size), (2 * r(9, size)).to(dtype), 1 + 0.2 * r(size)
    out = torch.full((9, size + 3), 7.0, dtype=dtype, device=dev)
    S.gated_norm(o.to(dev), z.to(dev), w.to(dev), 1e-2, 1, out, False, sigmoid=True)
    assert rel(out[:, :size], O.rms_norm(o.double(), 1e-2, w.double()) * torch.sigmoid(z.double())) < tol
    assert (out[:, size:] == 7).all()


# ------------------------------------------------------------------ routing
ROUTES = [(1, 1, 1, 1, 0), (6, 2, 3, 2, 1), (8, 3, 4, 1, 0), (8, 4, 2, 2, 2), (40, 8, 8, 4, 3), (64, 5, 64, 20, 0), (96, 6, 12, 3, 1),
          (256, 8, 8, 4, 1), (256, 20, 128, 100, 12), (300, 4, 100, 7, 0)]


@pytest.mark.parametrize("e,top,groups,keep,always", ROUTES)
def test_routing_by_groups(dev, e, top, groups, keep, always):
    if top > keep * (e // groups):
        top = keep * (e // groups)
    r, t = rand(e), 53
    z = 1.5 * r(t, e)
    i = lambda *s: torch.zeros(*s, dtype=torch.int32, device=dev)         # noqa: E731
    rt = R.Routing(i(t, top + always), torch.zeros(t, top + always, device=dev), None, i(e + always), i(e + always + 1),
                   i(t, top + always))
    g = R.RouteGroups(groups, keep, 1.7, always)
    R.route_grouped(z.to(dev), g, rt)
    spec = {"experts": e, "top": top, "scale": 1.7, "groups": {"count": groups, "keep": keep}}
    idx, wt = O.route(torch.eye(e, dtype=D), spec, z.double())
    got, order = rt.idx[:, :top].cpu().long().sort(1)
    want, back = idx.sort(1)
    assert torch.equal(got, want)
    assert rel(rt.weights[:, :top].cpu().gather(1, order), wt.gather(1, back)) < 1e-6
    assert torch.equal(rt.idx[:, top:].cpu(), torch.arange(e, e + always).expand(t, -1).int()) and (rt.weights[:, top:] == 1).all()
    count = torch.cat([torch.bincount(got.reshape(-1), minlength=e), torch.full((always,), t)])
    assert torch.equal(rt.offsets.cpu().long(), torch.cat([torch.zeros(1, dtype=torch.long), count.cumsum(0)]))
    h = r(t, 16)
    xs = torch.full((t * (top + always), 16), 9.0, device=dev)
    R.route_scatter(h.to(dev), rt, xs, always)
    rows = rt.row_of_pair.cpu().long()
    assert sorted(rows.reshape(-1).tolist()) == list(range(t * (top + always)))
    assert torch.equal(xs.cpu()[rows], h[:, None].expand(-1, top + always, -1))
    off = rt.offsets.cpu().long()
    assert ((rows >= off[rt.idx.cpu().long()]) & (rows < off[rt.idx.cpu().long() + 1])).all()
    for b in (1, 3, 6):                                   # the decode form: logits and choice in one launch
        w = fpad(r(e, 40) / 3, (0, 0)).to(BF)
        x, ticket = r(b, 40), i(1)
        rd = R.Routing(i(b, top + always), torch.zeros(b, top + always, device=dev), None, i(e + always), i(e + always + 1), i(b, top))
        for _ in range(2):                                # the ticket is left clean
            R.grouped_router(x.to(dev), w.to(dev), g, torch.empty(b, e, device=dev), ticket, rd)
        idx, wt = O.route(w.double(), spec, x.double())
        got, order = rd.idx[:, :top].cpu().long().sort(1)
        want, back = idx.sort(1)
        assert torch.equal(got, want) and rel(rd.weights[:, :top].cpu().gather(1, order), wt.gather(1, back)) < 1e-5
        assert torch.equal(rd.idx[:, top:].cpu(), torch.arange(e, e + always).expand(b, -1).int()) and int(ticket) == 0


FFS = [GroupedFfSpec(6, 2, 40, 3, 2, 1.5, 56), GroupedFfSpec(4, 1, 24, 1, 1, 0.5, 200), GroupedFfSpec(3, 3, 64, 1, 1, 2.0, 64),
       GroupedFfSpec(8, 3, 33, 4, 3, 1.0, 0), GroupedFfSpec(2, 1, 8, 1, 1, 1.0, 300)]


@pytest.mark.parametrize("dtype,tol", [(F32, 5e-6), (BF, 1e-2)])
@pytest.mark.parametrize("f", FFS, ids=lambda f: f"{f.experts}-{f.top}-{f.ff}-{f.shared}")
@pytest.mark.parametrize("t", [1, 3, 70])
def test_routed_and_shared_feed_forward(dev, dtype, tol, f, t):
    """The layer's kernels for a batch, and (bf16, few rows) the decode form."""
    cfg, tensors = one_layer(LIGHT[0], f, 44, seed=7)
    tensors = {k: v.to(dtype).float() for k, v in tensors.items()}
    model = M.NizoraxModel(M.build_weights(cfg, tensors, dev, dtype))
    fw, h = model.w.layers[0].mlp, padded(rand(t)(t, 44), dev, dtype)
    c = StepContext(t, Buffers(max(t, 8), dev), None, None, None, None, None, None)
    rt = model.routing(fw, c)
    R.route_grouped(model.router_logits(fw, h, c), model.groups(fw), rt)
    y = model.expert_rows(fw, h, rt, c)
    got = (rt.weights.double()[:, :, None] * y.double()[rt.row_of_pair.long()]).sum(1)[:, :44]
    mlp = {k[7:]: v.double() for k, v in tensors.items() if k.startswith("l0.mlp.")}
    want = O.expert_mix(mlp, f.to_json(), h[:, :44].double().cpu())
    assert rel(got, want) < tol
    if dtype == BF and t <= 3:
        eng = SandwichDecode(model, model.new_cache(4, max_seqs=4), max_batch=3, use_graph=False)
        out = torch.full((t, 48), 7.0, device=dev)
        eng._feed_forward(fw, h.float(), out, c)
        assert rel(out[:, :44], want) < 6e-3 and not out[:, 44:].any()


# ------------------------------------------------------------------ the model
def odd_cfg():
    """Widths that are not multiples of eight, single heads and groups, layers without feed-forward, top equal to the
    experts, one expert, no window, no rotation, a loop at the end; every constant different from layer to layer."""
    A, G, X, T = DifferentialAttentionSpec, LightningSpec, GroupedFfSpec, SandwichLayerSpec
    return NizoraxConfig(83, 100, [
        T(A(2, 1, 20, 36, 0.3, RotarySpec(50.0, 0), 0.6, 1), X(3, 3, 50, 1, 1, 0.7, 30)),
        T(G(1, 72, 36, [0.9]), None),
        T(A(5, 5, 12, 20, 0.25, RotarySpec(700.0, 2, LLAMA), 0.1, 0), X(1, 1, 33, 1, 1, 1.0, 100)),
        T(A(9, 1, 40, 72, 0.12, RotarySpec(1e6, 40, LLAMA), 0.8, 65), None),
        T(G(5, 9, 13, [0.1, 0.5, 0.9, 1.0, 0.0]), PolyNormFfSpec(33))],
        1e-3, 0.7, 1.3, taps=5, loop=LoopSpec(3, 5, 3)).validate()


def wide_cfg():
    """Head sizes outside the tensor-core attention kernels, a big state, one tap, everything in a loop."""
    A, G, T = DifferentialAttentionSpec, LightningSpec, SandwichLayerSpec
    return NizoraxConfig(65, 44, [
        T(A(2, 1, 136, 20, 0.1, RotarySpec(1e3, 64), 0.3, 33), PolyNormFfSpec(30)),
        T(G(1, 144, 300, [0.97]), GroupedFfSpec(4, 2, 24, 2, 1, 3.0, 0)),
        T(A(1, 1, 24, 264, 0.2, RotarySpec(1e3, 24), 0.5, 0), None)], 1e-4, 2.0, 0.5, taps=1, loop=LoopSpec(0, 3, 2)).validate()


def plain_cfg():
    """No loop; every layer of the kind the mat-vec decode form takes."""
    A, G, T = DifferentialAttentionSpec, LightningSpec, SandwichLayerSpec
    return NizoraxConfig(120, 72, [
        T(A(8, 2, 64, 128, 0.125, RotarySpec(1e4, 32, LLAMA), 0.4, 40), GroupedFfSpec(12, 3, 48, 4, 2, 1.2, 96)),
        T(G(4, 32, 32, [0.6, 0.9, 0.97, 0.999]), PolyNormFfSpec(100))], 1e-6, 4.0, 1.0, taps=4).validate()


CFGS = {"tiny": M.nizorax_tiny, "odd": odd_cfg, "wide": wide_cfg, "plain": plain_cfg}
TOL = {F32: 3e-5, BF: 0.2}


def settled(cfg, tensors):
    """Routers whose choice is far from close (bf16 rounding would flip close ones; the 32-bit runs and the routing tests
    above leave it to the logits): the norm's bias lifts every channel, the router reads the lift."""
    out, r = dict(tensors), rand(3)
    for i, l in enumerate(cfg.layers):
        if isinstance(l.mlp, GroupedFfSpec):
            z = torch.linspace(-2.5, 2.5, l.mlp.experts)[torch.randperm(l.mlp.experts, generator=torch.Generator().manual_seed(i))]
            out[f"l{i}.norm2.b"] = (tensors[f"l{i}.norm2.b"].float() + 2.0).to(BF)
            out[f"l{i}.mlp.router"] = ((z[:, None] / 2 + 0.05 * r(l.mlp.experts, cfg.width)) / cfg.width).to(BF)
    return out


class Bench:
    """A random model with its plain counterpart; prompts' logits are computed once."""

    def __init__(self, dev, name, dtype):
        self.cfg = CFGS[name]()
        self.tensors = M.random_tensors(self.cfg, 11)
        if dtype == BF:
            self.tensors = settled(self.cfg, self.tensors)
        self.model = M.NizoraxModel(M.build_weights(self.cfg, self.tensors, dev, dtype))
        self.dtype, self._ref, self._w = dtype, {}, {k: v.double() for k, v in self.tensors.items()}

    def tokens(self, n, seed):
        return torch.randint(0, self.cfg.vocab_size, (n,), generator=torch.Generator().manual_seed(seed)).tolist()

    def ref(self, toks):
        key = tuple(toks)
        if key not in self._ref:
            self._ref[key] = O.forward(self.cfg.to_json(), self._w, toks)
        return self._ref[key]

    def engine(self, blocks=80, batch=4, **kw):
        return ServingEngine(self.model, blocks, SchedulerConfig(max_batch_size=batch, **kw))

    def close(self, got, want):
        want = want.double().cpu()
        d = got.double().cpu() - want
        err = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
        return float(err.max()) < TOL[self.dtype] and (self.dtype == F32 or len(err) < 8 or float(err.median()) < 0.05)


@pytest.fixture(scope="module", params=[(n, d) for n in CFGS for d in (F32, BF)], ids=lambda p: f"{p[0]}-{str(p[1])[6:]}")
def bench(request):
    return Bench(torch.device("cuda:0"), *request.param)


def test_layers_one_by_one(bench):
    toks, want = bench.tokens(23, 1), []
    O.forward(bench.cfg.to_json(), bench._w, toks, lambda i, x: want.append(x))
    cache = bench.model.new_cache(4, max_seqs=1)
    cache.add_sequence(0)
    errs = []
    bench.model.forward_batch([Entry(0, toks, [22])], cache, observe=lambda li, x: errs.append(rel(x, want[li])))
    assert len(errs) == bench.cfg.num_layers and max(errs) < (2e-5 if bench.dtype == F32 else 5e-2)


@pytest.mark.parametrize("cuts", [[150], [2] * 20 + [110], [1] * 9 + [141], [16, 16, 15, 17, 3, 83], [64, 1, 64, 1, 1, 19],
                                  [129, 2, 2, 1, 1, 1, 14], [5] * 30], ids=str)
def test_a_prompt_in_portions(bench, cuts):
    toks = bench.tokens(150, 2)
    want = bench.ref(toks)
    eng = bench.engine()
    sid, at, got = eng.open_sequence(), 0, []
    for n in cuts:
        got.append(eng.run_entries([Entry(sid, toks[at:at + n], range(n))]))
        at += n
    assert at == 150 and bench.close(torch.cat(got), want)


def test_unequal_requests_together_and_slots_again(bench):
    """Four slots, ten requests of different lengths whose portions and decoded tokens share steps; pages and
    slots are used again, some requests pause, the pool is just large enough."""
    lens = [1, 2, 17, 70, 33, 5, 128, 16, 40, 64]
    reqs = [bench.tokens(n, 20 + i) for i, n in enumerate(lens)]
    eng = bench.engine(blocks=1 + (128 + 64 + 64 + 80) // 16)
    gen = torch.Generator().manual_seed(4)
    live, waiting, got, step = {}, list(range(10)), {i: [] for i in range(10)}, 0
    while live or waiting:
        while waiting and len(live) < 4:
            i = waiting.pop(0)
            live[i] = [eng.open_sequence(), 0]
        step += 1
        batch, order = [], []
        for i, (sid, at) in live.items():
            if (step + i) % 5 == 0 and len(live) > 1:
                continue                                  # this one pauses
            n = min(lens[i] - at, int(torch.tensor([1, 1, 2, 3, 13, 40])[torch.randint(6, (1,), generator=gen)]))
            batch.append(Entry(sid, reqs[i][at:at + n], range(n)))
            order.append((i, n))
        if not batch:
            continue
        out, lo = eng.run_entries(batch), 0
        for i, n in order:
            got[i].append(out[lo:lo + n].cpu())
            lo += n
            live[i][1] += n
            if live[i][1] == lens[i]:
                eng.close_sequence(live.pop(i)[0])
    for i, toks in enumerate(reqs):
        assert bench.close(torch.cat(got[i]), bench.ref(toks)), i


def test_result_does_not_depend_on_company_or_pages(bench):
    """One request alone on fresh pages, and in a crowd on used pages: the same up to rounding."""
    toks = bench.tokens(60, 40)
    a = bench.engine()
    s = a.open_sequence()
    alone = torch.cat([a.run_entries([Entry(s, toks[:50], range(50))])] +
                      [a.run_entries([Entry(s, [t], [0])]) for t in toks[50:]])
    b = bench.engine()
    junk = [b.open_sequence() for _ in range(3)]
    b.run_entries([Entry(j, bench.tokens(30 + j, 50 + j), ()) for j in junk])
    b.close_sequence(junk[1])
    s = b.open_sequence()
    crowd = [b.run_entries([Entry(junk[0], [3, 4], ()), Entry(s, toks[:50], range(50))])]
    for t in toks[50:]:
        crowd.append(b.run_entries([Entry(junk[2], [5], ()), Entry(s, [t], [0])]))
    assert worst_row(torch.cat(crowd), alone) < 2e-5 if bench.dtype == F32 else bench.close(torch.cat(crowd), alone)


def test_long_decoding(bench):
    toks = bench.tokens(310, 60)
    want = bench.ref(toks)
    eng = bench.engine()
    s = eng.open_sequence()
    got = [eng.run_entries([Entry(s, toks[:3], range(3))])]
    got += [eng.run_entries([Entry(s, [t], [0])]) for t in toks[3:]]
    assert bench.close(torch.cat(got), want)


@pytest.mark.parametrize("rows", [1, 3, 5, 16])
def test_decode_engine_buckets(bench, rows):
    """The captured step at several batch sizes (mat-vec and GEMM forms, idle rows), graph and eager; recording a
    step leaves no trace in the recurrent state, and rows keep their own."""
    prompts = [bench.tokens(4 + 7 * i % 40, 70 + i) for i in range(rows)]
    for use_graph in (True, False):
        cache = bench.model.new_cache(120, max_seqs=16)
        eng = SandwichDecode(bench.model, cache, max_batch=16, use_graph=use_graph)
        assert eng.fused == (bench.dtype == BF and bench.cfg.vocab_size != 65)
        for i, p in enumerate(prompts):
            cache.add_sequence(i)
            bench.model.prefill(torch.tensor(p[:-3]), cache, i)
        eng.bind(list(range(rows)), [p[-3] for p in prompts])
        eng.reserve(3)
        got = []
        for k in (-2, -1, 0):
            eng.step()
            got.append(eng.logits[:rows].clone())
            if k:
                eng.set_next_tokens([p[k] for p in prompts])
        for j in range(3):
            want = torch.stack([bench.ref(p)[j - 3] for p in prompts])
            assert bench.close(got[j], want), (use_graph, j)
        assert eng.launches_per_step > 0


def test_captured_decoding_over_a_window(bench):
    """Sixty captured steps in both forms: keys leave the windows, convolutions and states run on."""
    toks = bench.tokens(80, 33)
    want = bench.ref(toks)
    for rows in (1, 4):
        cache = bench.model.new_cache(40, max_seqs=4)
        eng = SandwichDecode(bench.model, cache, max_batch=4)
        for i in range(rows):
            cache.add_sequence(i)
            bench.model.prefill(torch.tensor(toks[:20]), cache, i)
        eng.bind(list(range(rows)), [toks[20]] * rows)
        eng.reserve(60)
        got = []
        for t in range(20, 80):
            eng.step()
            got.append(eng.logits[:rows].clone())
            if t < 79:
                eng.set_next_tokens([toks[t + 1]] * rows)
        for i in range(rows):
            assert bench.close(torch.stack([g[i] for g in got]), want[20:]), (rows, i)


def test_fork_copies_the_state(bench):
    toks = bench.tokens(40, 3)
    cache = bench.model.new_cache(20, max_seqs=3)
    cache.add_sequence(0)
    bench.model.prefill(torch.tensor(toks[:30]), cache, 0)
    cache.fork(0, 1)
    a = bench.model.forward_batch([Entry(1, toks[30:], range(10)), Entry(0, [1, 2, 3], ())], cache)
    assert bench.close(a, bench.ref(toks)[30:])


def _check_greedy(bench, prompt, got):
    """Every chosen token is the plain model's, or within rounding of its best logit."""
    hist = list(prompt)
    for t in got:
        lg = bench.ref(hist)[-1]
        slack = (2e-4 if bench.dtype == F32 else 0.3) * float(lg.std())
        assert float(lg.max() - lg[t]) <= slack
        hist.append(t)


def test_greedy_generation_through_the_scheduler(bench):
    prompts = [bench.tokens(n, 90 + n) for n in (1, 19, 50, 3, 33, 16)]
    eng = bench.engine(batch=3, max_prefill_chunk=16)
    ids = [eng.submit(p, 5) for p in prompts]
    out = eng.run_until_done()
    for sid, p in zip(ids, prompts):
        assert len(out[sid]) == 5
        _check_greedy(bench, p, out[sid])
    p = prompts[1]
    got = bench.model.generate_greedy(torch.tensor(p), 5)
    assert len(got) == 5
    _check_greedy(bench, p, got)


def test_sampling_through_the_engine(bench):
    eng = ServingEngine(bench.model, 60, SchedulerConfig(max_batch_size=2, max_prefill_chunk=16),
                        SamplerConfig(temperature=0.8, top_k=5, seed=3))
    ids = [eng.submit(bench.tokens(20, 7), 6), eng.submit(bench.tokens(4, 8), 6)]
    out = eng.run_until_done()
    for sid, seed, n in zip(ids, (7, 8), (20, 4)):
        hist = bench.tokens(n, seed)
        for t in out[sid]:
            assert t in bench.ref(hist)[-1].topk(14).indices.tolist()
            hist.append(t)


def test_warm_up_and_other_entry_points(bench):
    eng = bench.engine(batch=2)
    eng.warm_up(prompt_len=5, new_tokens=2)
    assert eng.cache.manager.num_free_blocks() >= 70
    toks = bench.tokens(40, 5)
    assert bench.close(bench.model.forward(torch.tensor(toks)), bench.ref(toks))
    s = eng.open_sequence()                               # a slot the warm-up has used
    assert bench.close(eng.run_entries([Entry(s, toks, range(40))]), bench.ref(toks))


def test_command_line_generation_and_trace(tmp_path, dev):
    from rmlx_b200.cli.main import main
    b = Bench(dev, "odd", F32)
    M.save_checkpoint(str(tmp_path / "m"), b.cfg, b.tensors)
    prompt = [5, 9, 80, 3]
    out, real = io.StringIO(), sys.stdout
    sys.stdout = out
    try:
        assert main(["generate", "--model", str(tmp_path / "m"), "--prompt", "5,9,80,3", "--steps", "4",
                     "--dtype", "float32"]) == 0
    finally:
        sys.stdout = real
    toks = json.loads(out.getvalue().splitlines()[-1])["tokens"]
    assert len(toks) == 1 and len(toks[0]) == 4
    _check_greedy(b, prompt, toks[0])
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": prompt[:3], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": prompt[3:], "want": [0]},
                                     {"id": "y", "tokens": [1, 2], "want": [1, 0]}], "end": ["x", "y"]},
             {"step": 2, "entries": [{"id": "x", "tokens": [1, 2], "want": [1]}], "end": ["x"]}]
    (tmp_path / "o").mkdir()
    out, real_in = io.StringIO(), sys.stdin
    sys.stdin, sys.stdout = io.StringIO("".join(json.dumps(s) + "\n" for s in steps)), out
    try:
        assert main(["trace-run", "--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(tmp_path / "o"),
                     "--max-tokens", "128"]) == 0
    finally:
        sys.stdin, sys.stdout = real_in, real
    assert out.getvalue().split() == ["done", "0", "done", "1", "done", "2"] and not (tmp_path / "o" / "0.f32").exists()

    def read(name):
        data = (tmp_path / "o" / name).read_bytes()
        return torch.tensor(struct.unpack(f"<{len(data) // 4}f", data)).view(-1, b.cfg.vocab_size)

    want = torch.stack([b.ref(prompt)[-1], b.ref([1, 2])[1], b.ref([1, 2])[0]])
    assert worst_row(read("1.f32"), want) < TOL[F32] and worst_row(read("2.f32"), b.ref([1, 2])[1:]) < TOL[F32]
