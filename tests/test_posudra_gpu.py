"""Posudra on the GPU against the plain restatement in ``oracle/posudra.py``: every kernel alone, then the
model through its ragged batches, its decode engine, the serving engine and the command line, in 32-bit
(tight) and bf16."""
import math

import pytest
import torch
from oracle import posudra as O

from rmlx_b200.config import ParallelLayerSpec, PosudraConfig, SamplerConfig, SchedulerConfig, ScoredAttentionSpec
from rmlx_b200.models import posudra as M
from rmlx_b200.models.parallel_decode import ParallelBlockDecode
from rmlx_b200.models.ragged import Entry, query_tiles
from rmlx_b200.ops import parallel_block as P
from rmlx_b200.serve.engine import ServingEngine

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32


def rel(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    return float((got - want).norm() / want.norm().clamp_min(1e-30))


def worst_row(got, want):
    """Largest error of a row of logits (mean taken off) over the rms of the logits."""
    d = got.double().cpu() - want.double().cpu()
    d = d - d.mean(-1, keepdim=True)
    return float(d.pow(2).mean(-1).sqrt().max() / want.double().pow(2).mean().sqrt())


class Heads:
    """Random q / k / v of several sequences in pages, and the plain attention over them."""

    def __init__(self, dev, lens, hq, hkv, dk, dv, dtype=BF, seed=0, scale=None, cap=20.0, kscale=1.0):
        g = torch.Generator().manual_seed(seed)
        r = lambda *s: torch.randn(*s, generator=g)                       # noqa: E731
        self.hq, self.hkv, self.dk, self.dv, self.lens, self.dev, self.dtype = hq, hkv, dk, dv, lens, dev, dtype
        self.dkp, self.dvp = P.pad8(dk), P.pad8(dv)
        self.q = [r(n, hq, dk).to(dtype) for n in lens]
        self.k = [(r(n, hkv, dk) * kscale).to(dtype) for n in lens]
        self.v = [r(n, hkv, dv).to(dtype) for n in lens]
        self.scale, self.cap = scale or dk ** -0.5, cap
        self.temp, self.r1, self.r2 = r(hq).abs() + 0.5, 0.3 * r(hq).abs(), 0.2 * r(hq).abs()
        self.sink = r(hq)

    def mods(self, **kw):
        c = lambda t: t.to(self.dev, F32)                                 # noqa: E731
        d = dict(scale=self.scale, softcap=self.cap, temp=c(self.temp), r1=c(self.r1), r2=c(self.r2), sink=c(self.sink))
        d.update(kw)
        return P.ScoreMods(**d)

    def build(self):
        """Pages in shuffled order (page 0 stays reserved), zero padding as the cache keeps it."""
        npg = [(n + 15) // 16 for n in self.lens]
        order = torch.randperm(sum(npg), generator=torch.Generator().manual_seed(5)) + 1
        kc = torch.zeros(sum(npg) + 1, self.hkv, 16, self.dkp, dtype=self.dtype)
        vc = torch.zeros(sum(npg) + 1, self.hkv, 16, self.dvp, dtype=self.dtype)
        table = torch.zeros(len(self.lens), max(npg), dtype=torch.int32)
        at = 0
        for i, n in enumerate(self.lens):
            pages = order[at:at + npg[i]]
            at += npg[i]
            table[i, :npg[i]] = pages.int()
            for t in range(n):
                kc[pages[t // 16], :, t % 16, :self.dk] = self.k[i][t]
                vc[pages[t // 16], :, t % 16, :self.dv] = self.v[i][t]
        return kc.to(self.dev), vc.to(self.dev), table.to(self.dev)

    def padded_q(self, rows):
        """rows: (sequence, position) -> [R, Hq, dkp]."""
        q = torch.full((len(rows), self.hq, self.dkp), 0.0, dtype=self.dtype)
        for i, (s, t) in enumerate(rows):
            q[i, :, :self.dk] = self.q[s][t]
        return q.to(self.dev)

    def want(self, rows, window=0, **kw):
        outs = {}
        for s in {s for s, _ in rows}:
            d = lambda t: t.double()                                      # noqa: E731
            a = dict(temp=d(self.temp), r1=d(self.r1), r2=d(self.r2), sink=d(self.sink), cap=self.cap)
            a.update(kw)
            q, k, v = (d(x[s]).permute(1, 0, 2) for x in (self.q, self.k, self.v))
            k, v = O.repeat_groups(k, self.hq), O.repeat_groups(v, self.hq)
            if window:
                full = torch.zeros(q.shape[0], q.shape[1], self.dv, dtype=torch.float64)
                for t in range(q.shape[1]):
                    lo = max(0, t - window + 1)
                    full[:, t] = O.scored_attention(q[:, lo:t + 1], k[:, lo:t + 1], v[:, lo:t + 1], self.scale, a["temp"],
                                                    a["cap"], a["r1"], a["r2"], a["sink"])[:, -1]
                outs[s] = full
            else:
                outs[s] = O.scored_attention(q, k, v, self.scale, a["temp"], a["cap"], a["r1"], a["r2"], a["sink"])
        return torch.stack([outs[s][:, t] for s, t in rows])


SHAPES = [(4, 2, 32, 40), (6, 2, 72, 16), (8, 1, 128, 128), (2, 2, 20, 70), (3, 1, 128, 64), (40, 2, 64, 64)]


@pytest.mark.parametrize("shape", SHAPES, ids=str)
@pytest.mark.parametrize("lanes", [1, 2])
@pytest.mark.parametrize("cap", [20.0, 1.5])
def test_prompt_attention_ragged(dev, shape, lanes, cap):
    # cap 1.5: many scores beyond the polynomial's range
    h = Heads(dev, [2, 17, 130, 300], *shape, cap=cap)
    kc, vc, table = h.build()
    # portions that end their sequences: whole, whole, from 1, from 45
    starts = [0, 0, 1, 45]
    rows = [(s, t) for s, lo in enumerate(starts) for t in range(lo, h.lens[s])]
    q = h.padded_q(rows)
    lens = [n - lo for n, lo in zip(h.lens, starts)]
    firsts = [sum(lens[:i]) for i in range(4)]
    tiles = torch.tensor(query_tiles(firsts, lens, starts, [0, 1, 2, 3], 128 * lanes), dtype=torch.int32, device=dev)
    out = torch.full((len(rows), h.hq, h.dvp), 7.0, dtype=BF, device=dev)
    P.flash_prefill_scored(q, kc, vc, table, tiles, h.mods(), out, lanes=lanes)
    assert rel(out[..., :h.dv], h.want(rows)) < 6e-3
    assert not out[..., h.dv:].any()


@pytest.mark.parametrize("shape", SHAPES, ids=str)
@pytest.mark.parametrize("splits", [1, 3, 16])
def test_decode_attention_plain(dev, shape, splits):
    h = Heads(dev, [1, 15, 16, 17, 33, 257, 400], *shape, seed=1)
    kc, vc, table = h.build()
    rows = [(s, n - 1) for s, n in enumerate(h.lens)]
    q = h.padded_q(rows)
    pos = torch.tensor([n - 1 for n in h.lens], dtype=torch.int32, device=dev)
    out = torch.zeros(len(rows), h.hq, h.dvp, dtype=BF, device=dev)
    scr = P.ScoredDecodeScratch(len(rows), h.hq, h.hkv, h.dvp, splits, dev)
    for _ in range(2):                                    # the tickets are left clean
        P.flash_decode_scored(kc, vc, table, pos, h.mods(), out, scr, h.hq, h.dk, h.dv, q=q)
        assert rel(out[..., :h.dv], h.want(rows)) < 6e-3
    # a subset of the rows, the others untouched
    out.fill_(3.0)
    pick = torch.tensor([5, 1], dtype=torch.int32, device=dev)
    P.flash_decode_scored(kc, vc, table, pos, h.mods(), out, scr, h.hq, h.dk, h.dv, q=q, rows=pick)
    assert rel(out[[5, 1], :, :h.dv], h.want([rows[5], rows[1]])) < 6e-3 and (out[[0, 2, 3, 4, 6]] == 3.0).all()


@pytest.mark.parametrize("shape", SHAPES, ids=str)
def test_decode_attention_fused_norm_and_append(dev, shape):
    hq, hkv, dk, dv = shape
    g = torch.Generator().manual_seed(3)
    h = Heads(dev, [1, 16, 17, 200], *shape, seed=2)
    nq, nk, nv = hq * dk, hkv * dk, hkv * dv
    raw = torch.randn(4, nq + nk + nv + 3, generator=g)
    qw, kw = 1 + 0.3 * torch.randn(nq, generator=g), 1 + 0.3 * torch.randn(nk, generator=g)
    for s, n in enumerate(h.lens):                        # the restatement's view of the new token
        h.q[s][n - 1] = O.rms_norm(raw[s, :nq], qw, 1e-5).view(hq, dk).to(BF)
        h.k[s][n - 1] = O.rms_norm(raw[s, nq:nq + nk], kw, 1e-5).view(hkv, dk).to(BF)
        h.v[s][n - 1] = raw[s, nq + nk:nq + nk + nv].view(hkv, dv).to(BF)
    rows = [(s, n - 1) for s, n in enumerate(h.lens)]
    want_k, want_v, table = h.build()
    kc, vc = want_k.clone(), want_v.clone()
    for s, n in enumerate(h.lens):                        # the slot of the new token starts dirty
        page = int(table[s, (n - 1) // 16])
        kc[page, :, (n - 1) % 16, :dk] = 9.0
        vc[page, :, (n - 1) % 16, :dv] = -9.0
    pos = torch.tensor([n - 1 for n in h.lens], dtype=torch.int32, device=dev)
    for splits in (1, 5):
        out = torch.zeros(4, hq, h.dvp, dtype=BF, device=dev)
        scr = P.ScoredDecodeScratch(4, hq, hkv, h.dvp, splits, dev)
        P.flash_decode_scored(kc, vc, table, pos, h.mods(), out, scr, hq, dk, dv, raw=raw.to(dev), q_w=qw.to(dev),
                              k_w=kw.to(dev), eps=1e-5)
        assert rel(out[..., :dv], h.want(rows)) < 6e-3
        assert rel(kc, want_k) < 2e-3 and torch.equal(vc, want_v)


@pytest.mark.parametrize("dtype,tol", [(F32, 2e-6), (BF, 4e-3)])
@pytest.mark.parametrize("shape", [(4, 2, 20, 40), (2, 1, 200, 264), (3, 3, 8, 130)], ids=str)
def test_attention_any(dev, dtype, tol, shape):
    h = Heads(dev, [1, 31, 32, 33, 150], *shape, dtype=dtype, seed=4)
    kc, vc, table = h.build()
    rows = [(s, t) for s, n in enumerate(h.lens) for t in range(n)]
    pos = torch.tensor([t for _, t in rows], dtype=torch.int32, device=dev)
    seq = torch.tensor([s for s, _ in rows], dtype=torch.int32, device=dev)
    out = torch.empty(len(rows), h.hq, h.dvp, dtype=dtype, device=dev)
    P.attention_any(h.padded_q(rows), kc, vc, table, pos, seq, h.mods(), out)
    assert rel(out[..., :h.dv], h.want(rows)) < tol
    P.attention_any(h.padded_q(rows), kc, vc, table, pos, seq, h.mods(), out, window=9)
    assert rel(out[..., :h.dv], h.want(rows, window=9)) < tol


def _all_three(h, rows, starts, dev, mods, window=0):
    """The same rows (sequences' tails from ``starts``) through every bf16 attention kernel."""
    kc, vc, table = h.build()
    q = h.padded_q(rows)
    lens = [n - lo for n, lo in zip(h.lens, starts)]
    firsts = [sum(lens[:i]) for i in range(len(lens))]
    slots = list(range(len(lens)))
    pos = torch.tensor([t for _, t in rows], dtype=torch.int32, device=dev)
    seq = torch.tensor([s for s, _ in rows], dtype=torch.int32, device=dev)
    new = lambda: torch.zeros(len(rows), h.hq, h.dvp, dtype=BF, device=dev)     # noqa: E731
    outs = {}
    for lanes in (1, 2):
        tiles = torch.tensor(query_tiles(firsts, lens, starts, slots, 128 * lanes), dtype=torch.int32, device=dev)
        outs[f"prompt{lanes}"] = P.flash_prefill_scored(q, kc, vc, table, tiles, mods, new(), window=window, lanes=lanes)
    for splits in (1, 4):
        scr = P.ScoredDecodeScratch(len(rows), h.hq, h.hkv, h.dvp, splits, dev)
        outs[f"decode{splits}"] = P.flash_decode_scored(kc, vc, table, pos, mods, new(), scr, h.hq, h.dk, h.dv, q=q,
                                                        table_rows=seq, window=window)
    outs["any"] = P.attention_any(q, kc, vc, table, pos, seq, mods, new(), window=window)
    return {n: o[..., :h.dv] for n, o in outs.items()}


def test_a_far_key_stands_out_in_every_kernel(dev):
    """One key (on a page border, in the first page, far back) is aligned with one query so that its
    weight is large despite hundreds of others; leaving it out, or seeing one key too many, shows."""
    h = Heads(dev, [700], 4, 2, 48, 56, seed=6, cap=30.0)
    h.r1.fill_(0.05)
    h.sink.fill_(-2.0)
    for t, j in ((650, 0), (660, 15), (670, 16), (699, 640), (680, 680), (690, 127)):
        q = h.q[0][t].float()
        h.k[0][j] = (q.view(2, 2, 48)[:, 0] * 2.5).to(BF)
    rows = [(0, t) for t in range(600, 700)]
    want = h.want(rows)
    # on the CPU: the weight of each planted key is dominant, so a lost key is far outside the tolerance
    lost = Heads(dev, [700], 4, 2, 48, 56, seed=6, cap=30.0)
    lost.q, lost.v, lost.k = h.q, h.v, [h.k[0].clone()]
    lost.r1, lost.sink = h.r1, h.sink
    lost.k[0][[0, 15, 16, 127]] = 0
    assert rel(lost.want(rows)[[50, 60, 70, 90]], want[[50, 60, 70, 90]]) > 0.3
    for name, got in _all_three(h, rows, [600], dev, h.mods()).items():
        assert rel(got, want) < 8e-3, name
        for i in (50, 60, 70, 80, 90, 99):
            assert rel(got[i], want[i]) < 1.5e-2, (name, i)


def test_window_edges_in_every_kernel(dev):
    h = Heads(dev, [200], 2, 1, 64, 32, seed=7)
    rows = [(0, t) for t in range(100, 200)]
    for window in (1, 16, 33):
        for edge, key in (("in", 150 - window + 1), ("out", 150 - window)):
            h.k[0][key] = (h.q[0][150].float()[0] * 3).to(BF)
        want = h.want(rows, window=window)
        for name, got in _all_three(h, rows, [100], dev, h.mods(), window=window).items():
            assert rel(got, want) < 8e-3, (name, window)
            assert rel(got[50], want[50]) < 1.5e-2, (name, window)


@pytest.mark.parametrize("part", ["temp", "bias", "cap", "sink"])
def test_each_modifier_alone_in_every_kernel(dev, part):
    h = Heads(dev, [90, 33], 4, 2, 40, 24, seed=8, scale=0.3)
    h.sink.mul_(3)
    rows = [(0, t) for t in range(60, 90)] + [(1, t) for t in range(33)]
    big, one = 1e9, torch.ones(4, dtype=torch.float64)
    off = dict(temp=one, r1=0 * one, r2=0 * one, sink=-big * one, cap=1e6)
    kw = dict(temp=None, r1=None, r2=None, sink=None, softcap=0.0)
    plain = h.want(rows, **off)
    if part == "temp":
        off["temp"], kw["temp"] = h.temp.double(), h.mods().temp
    elif part == "bias":
        off["r1"], off["r2"] = h.r1.double(), h.r2.double()
        kw["r1"], kw["r2"] = h.mods().r1, h.mods().r2
    elif part == "cap":
        off["cap"] = kw["softcap"] = 1.0
    else:
        off["sink"], kw["sink"] = h.sink.double(), h.mods().sink
    want = h.want(rows, **off)
    assert rel(want, plain) > 0.03                        # the part matters on these inputs
    for name, got in _all_three(h, rows, [60, 0], dev, h.mods(**kw)).items():
        assert rel(got, want) < 8e-3, name
    for name, got in _all_three(h, rows, [60, 0], dev, h.mods(temp=None, r1=None, r2=None, sink=None, softcap=0.0)).items():
        assert rel(got, plain) < 8e-3, name


def test_saturated_scores_and_large_sink_in_every_kernel(dev):
    """Scores far beyond the cap next to small ones, and a sink just under the cap."""
    h = Heads(dev, [150], 2, 1, 32, 32, seed=9, cap=12.0, kscale=20.0)
    h.sink.fill_(11.5)
    rows = [(0, t) for t in range(20, 150)]
    want = h.want(rows)
    assert rel(h.want(rows, sink=torch.full((2,), -1e9, dtype=torch.float64)), want) > 0.1
    for name, got in _all_three(h, rows, [20], dev, h.mods()).items():
        assert rel(got, want) < 1e-2, name


# ------------------------------------------------------------------ projections and row kernels
@pytest.mark.parametrize("dtype,tol", [(F32, 3e-6), (BF, 5e-3)])
@pytest.mark.parametrize("t,k,n_raw,ff", [(1, 24, 32, 8), (130, 104, 96, 200), (77, 512, 288, 0), (300, 264, 32, 1000)])
def test_in_and_out_projections(dev, dtype, tol, t, k, n_raw, ff):
    g = torch.Generator().manual_seed(t)
    r = lambda *s: torch.randn(*s, generator=g)                           # noqa: E731
    h, w = r(t, k).to(dtype), (r(n_raw + ff, k) / k ** 0.5).to(dtype)
    raw = torch.empty(t, n_raw, dtype=dtype, device=dev)
    act = torch.empty(t, ff, dtype=dtype, device=dev) if ff else None
    p, q = torch.tensor(0.4).double(), torch.tensor(-0.6).double()
    ap, an = float(torch.nn.functional.softplus(p)), 0.5 + float(torch.nn.functional.softplus(q))
    P.in_proj(h.to(dev), w.to(dev), n_raw, ap, an, raw, act)
    full = h.double() @ w.double().T
    assert rel(raw, full[:, :n_raw]) < tol
    if ff:
        assert rel(act, O.xielu(full[:, n_raw:], p, q)) < tol
    # the two output projections into the residual
    k1 = 40
    a, wo, wd = r(t, k1).to(dtype), r(k, k1).to(dtype), (r(k, ff).to(dtype) if ff else None)
    ls1, ls2, x = r(k), r(k), r(t, k)
    xd = x.to(dev)
    act_in = r(t, ff).to(dtype) if ff else None
    P.out_proj_add(a.to(dev), wo.to(dev), ls1.to(dev), None if not ff else act_in.to(dev), None if not ff else wd.to(dev),
                   ls2.to(dev) if ff else None, xd)
    want = x.double() + ls1.double() * (a.double() @ wo.double().T)
    if ff:
        want = want + ls2.double() * (act_in.double() @ wd.double().T)
    assert rel(xd, want) < 3e-6


@pytest.mark.parametrize("b", [1, 3, 4, 6])
@pytest.mark.parametrize("ff", [0, 72])
def test_decode_projections(dev, b, ff):
    g = torch.Generator().manual_seed(b)
    r = lambda *s: torch.randn(*s, generator=g)                           # noqa: E731
    d, k, n_raw = 100, 104, 64
    x = torch.zeros(b, k)
    x[:, :d] = r(b, d) * 3
    nw, w = torch.zeros(k), torch.zeros(n_raw + ff, k)
    nw[:d], w[:, :d] = 1 + 0.2 * r(d), r(n_raw + ff, d) / 10
    w = w.to(BF)
    raw = torch.empty(b, n_raw, device=dev)
    act = torch.empty(b, ff, dtype=BF, device=dev) if ff else None
    p, q = torch.tensor(-0.3).double(), torch.tensor(0.2).double()
    sp = torch.nn.functional.softplus
    P.norm_in_proj(x.to(dev), nw.to(dev), 1e-4, d, w.to(dev), n_raw, float(sp(p)), 0.5 + float(sp(q)), raw, act)
    z = O.rms_norm(x[:, :d].double(), nw[:d].double(), 1e-4) @ w[:, :d].double().T
    assert rel(raw, z[:, :n_raw]) < 2e-6
    if ff:
        assert rel(act, O.xielu(z[:, n_raw:], p, q)) < 4e-3
    a, wo = r(b, 48).to(BF), r(k, 48).to(BF)
    wd, ai = (r(k, ff).to(BF), r(b, ff).to(BF)) if ff else (None, None)
    ls1, ls2, xd = r(k), r(k), x.to(dev)
    P.gemv_out_add(a.to(dev), wo.to(dev), ls1.to(dev), None if not ff else ai.to(dev), None if not ff else wd.to(dev),
                   ls2.to(dev), xd)
    want = x.double() + ls1.double() * (a.double() @ wo.double().T)
    if ff:
        want = want + ls2.double() * (ai.double() @ wd.double().T)
    assert rel(xd, want) < 2e-6


@pytest.mark.parametrize("dtype,tol", [(F32, 1e-6), (BF, 4e-3)])
@pytest.mark.parametrize("hq,hkv,dk,dv", [(3, 1, 20, 10), (6, 3, 72, 40)])
def test_norms_append_and_embedding(dev, dtype, tol, hq, hkv, dk, dv):
    g = torch.Generator().manual_seed(1)
    r = lambda *s: torch.randn(*s, generator=g)                           # noqa: E731
    t, page = 37, 16
    nq, nk, nv = hq * dk, hkv * dk, hkv * dv
    raw = r(t, (nq + nk + nv + 31) // 32 * 32).to(dtype)
    qw, kw = 1 + 0.2 * r(nq), 1 + 0.2 * r(nk)
    kc = torch.zeros(9, hkv, page, P.pad8(dk), dtype=dtype, device=dev)
    vc = torch.zeros(9, hkv, page, P.pad8(dv), dtype=dtype, device=dev)
    table = torch.tensor([[4, 2, 8], [7, 1, 3]], dtype=torch.int32, device=dev)
    seq = [0] * 17 + [1] * 20
    pos = list(range(14, 31)) + list(range(20))
    q = torch.full((t, hq, P.pad8(dk)), 5.0, dtype=dtype, device=dev)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)        # noqa: E731
    P.qk_norm_append(raw.to(dev), qw.to(dev), kw.to(dev), 1e-3, q, kc, vc, table, i32(pos), i32(seq), hq, dk, dv)
    d = raw.double()
    assert rel(q[..., :dk], O.rms_norm(d[:, :nq], qw.double(), 1e-3).view(t, hq, dk)) < tol and not q[..., dk:].any()
    blk = [int(table[s, p // page]) for s, p in zip(seq, pos)]
    off = [p % page for p in pos]
    assert rel(kc[blk, :, off, :dk], O.rms_norm(d[:, nq:nq + nk], kw.double(), 1e-3).view(t, hkv, dk)) < tol
    assert torch.equal(vc[blk, :, off, :dv].cpu(), raw[:, nq + nk:nq + nk + nv].view(t, hkv, dv))
    assert not kc[..., dk:].any() and not vc[..., dv:].any() and not kc[[0, 5, 6]].any()
    table_e = r(50, 30).to(dtype)
    ids = torch.randint(0, 50, (11,), generator=g)
    x = torch.full((11, 32), 9.0, device=dev)
    P.embed_scaled(table_e.to(dev), ids.int().to(dev), 1.7, x)
    assert rel(x[:, :30], O.embed(table_e.double(), ids, 1.7)) < 1e-7 and not x[:, 30:].any()
    nw = torch.zeros(32)
    nw[:30] = 1 + r(30)
    out = torch.empty(11, 32, dtype=dtype, device=dev)
    P.rms_norm_f32(x, nw.to(dev), 1e-2, out, 30)
    assert rel(out[:, :30], O.rms_norm(x[:, :30].double().cpu(), nw[:30].double(), 1e-2)) < tol and not out[:, 30:].any()


# ------------------------------------------------------------------ the model
def wide_cfg():
    """Head sizes outside the tensor-core attention kernels, odd widths, one layer."""
    return PosudraConfig(65, 44, [ParallelLayerSpec(ScoredAttentionSpec(2, 1, 136, 20, 0.1, 9.0), 30)], 1e-4, 0.7).validate()


def odd_cfg():
    """Unequal layers: width 100, a single head, groups, no feed-forward somewhere, no cap equal to another."""
    A, L = ScoredAttentionSpec, ParallelLayerSpec
    return PosudraConfig(211, 100, [L(A(1, 1, 16, 8, 0.3, 11.0), 60), L(A(5, 5, 12, 20, 0.2, 30.0), 0),
                                    L(A(12, 2, 64, 64, 0.125, 25.0), 250), L(A(4, 2, 128, 96, 0.07, 40.0), 8)],
                         1e-3, 5.0).validate()


CFGS = {"tiny": M.posudra_tiny, "wide": wide_cfg, "odd": odd_cfg}
TOL = {F32: 2e-5, BF: 4e-2}


class Bench:
    """A random model with its plain counterpart; prompts' logits are computed once."""

    def __init__(self, dev, name, dtype):
        self.cfg = CFGS[name]()
        self.tensors = M.random_tensors(self.cfg, 11)
        self.model = M.PosudraModel(M.build_weights(self.cfg, self.tensors, dev, dtype))
        self.dtype, self._ref = dtype, {}

    def tokens(self, n, seed):
        return torch.randint(0, self.cfg.vocab_size, (n,), generator=torch.Generator().manual_seed(seed)).tolist()

    def ref(self, toks):
        key = tuple(toks)
        if key not in self._ref:
            self._ref[key] = O.forward(self.cfg.to_json(), self.tensors, toks)
        return self._ref[key]

    def engine(self, blocks=80, batch=4, **kw):
        return ServingEngine(self.model, blocks, SchedulerConfig(max_batch_size=batch, **kw))


@pytest.fixture(scope="module", params=[(n, d) for n in CFGS for d in (F32, BF)],
                ids=lambda p: f"{p[0]}-{str(p[1])[6:]}")
def bench(request):
    return Bench(torch.device("cuda:0"), *request.param)


def test_layers_one_by_one(bench):
    toks = bench.tokens(23, 1)
    _, want = O.forward(bench.cfg.to_json(), bench.tensors, toks, want_layers=True)
    cache = bench.model.new_cache(4, max_seqs=1)
    cache.add_sequence(0)
    errs = []
    bench.model.forward_batch([Entry(0, toks, [22])], cache, observe=lambda li, x: errs.append(rel(x, want[li])))
    assert len(errs) == bench.cfg.num_layers and max(errs) < TOL[bench.dtype]


@pytest.mark.parametrize("cuts", [[150], [2] * 20 + [110], [1] * 9 + [141], [16, 16, 15, 17, 3, 83], [64, 1, 64, 1, 1, 19],
                                  [129, 2, 2, 1, 1, 1, 14]], ids=str)
def test_a_prompt_in_portions(bench, cuts):
    toks = bench.tokens(150, 2)
    want = bench.ref(toks)
    eng = bench.engine()
    sid, at, got = eng.open_sequence(), 0, []
    for n in cuts:
        got.append(eng.run_entries([Entry(sid, toks[at:at + n], range(n))]))
        at += n
    assert at == 150 and worst_row(torch.cat(got), want) < TOL[bench.dtype]


def test_unequal_requests_together_and_slots_again(bench):
    """Four slots, ten requests of different lengths whose portions and decoded tokens share steps;
    pages and slots are used again, some requests pause, the pool is just large enough."""
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
        assert worst_row(torch.cat(got[i]), bench.ref(toks)) < TOL[bench.dtype], i


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
    assert worst_row(torch.cat(crowd), alone) < (1e-5 if bench.dtype == F32 else 3e-2)


def test_long_decoding(bench):
    toks = bench.tokens(310, 60)
    want = bench.ref(toks)
    eng = bench.engine()
    s = eng.open_sequence()
    got = [eng.run_entries([Entry(s, toks[:3], range(3))])]
    got += [eng.run_entries([Entry(s, [t], [0])]) for t in toks[3:]]
    assert worst_row(torch.cat(got), want) < TOL[bench.dtype]


@pytest.mark.parametrize("rows", [1, 3, 5, 16])
def test_decode_engine_buckets(bench, rows):
    """The captured step at several batch sizes (mat-vec and GEMM forms, idle rows), graph and eager."""
    prompts = [bench.tokens(4 + 7 * i % 40, 70 + i) for i in range(rows)]
    for use_graph in (True, False):
        cache = bench.model.new_cache(120, max_seqs=16)
        eng = ParallelBlockDecode(bench.model, cache, max_batch=16, use_graph=use_graph)
        for i, p in enumerate(prompts):
            cache.add_sequence(i)
            bench.model.prefill(torch.tensor(p[:-1]) if len(p) > 1 else torch.tensor(p), cache, i)
        eng.bind(list(range(rows)), [p[-1] for p in prompts])
        eng.reserve(1)
        eng.step()
        for i, p in enumerate(prompts):
            assert worst_row(eng.logits[i:i + 1], bench.ref(p)[-1:]) < TOL[bench.dtype], (use_graph, i)
        assert eng.launches_per_step > 0


def _check_greedy(bench, prompt, got):
    """Every chosen token is the plain model's, or within rounding of its best logit."""
    hist = list(prompt)
    for t in got:
        lg = bench.ref(hist)[-1]
        slack = (1e-4 if bench.dtype == F32 else 0.15) * float(lg.std())
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
            assert t in bench.ref(hist)[-1].topk(12).indices.tolist()
            hist.append(t)


def test_cached_prefix_is_reused(bench):
    eng = ServingEngine(bench.model, 60, SchedulerConfig(max_batch_size=2, max_prefill_chunk=32), use_prefix_cache=True)
    head = bench.tokens(48, 30)
    prompts = [head + bench.tokens(9, 31), head + bench.tokens(14, 32)]
    for p, ran in zip(prompts, (57, 14)):
        before = eng.prefill_tokens
        sid = eng.submit(p, 4)
        _check_greedy(bench, p, eng.run_until_done()[sid])
        eng.step()
        assert eng.prefill_tokens - before == ran


def test_warm_up_and_other_entry_points(bench):
    eng = bench.engine(batch=2)
    eng.warm_up(prompt_len=5, new_tokens=2)
    assert eng.cache.manager.num_free_blocks() >= 70
    toks = bench.tokens(12, 5)
    assert worst_row(bench.model.forward(torch.tensor(toks)), bench.ref(toks)) < TOL[bench.dtype]
    with pytest.raises(ValueError):
        bench.model.new_cache(4, kv_quant="q8")


def test_command_line_generation_and_trace(tmp_path, dev):
    import io
    import json
    import struct
    import sys
    from rmlx_b200.cli.main import main
    cfg = odd_cfg()
    tensors = M.random_tensors(cfg, 11)
    M.save_checkpoint(str(tmp_path / "m"), cfg, tensors)
    prompt = [5, 9, 100, 3]
    b = Bench(dev, "odd", F32)
    out = io.StringIO()
    real, sys.stdout = sys.stdout, out
    try:
        assert main(["generate", "--model", str(tmp_path / "m"), "--prompt", "5,9,100,3", "--steps", "4",
                     "--dtype", "float32"]) == 0
    finally:
        sys.stdout = real
    toks = json.loads(out.getvalue().splitlines()[-1])["tokens"]
    assert len(toks) == 1 and len(toks[0]) == 4
    _check_greedy(b, prompt, toks[0])
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": prompt[:3], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": prompt[3:], "want": [0]},
                                     {"id": "y", "tokens": [1, 2], "want": [1, 0]}], "end": ["x", "y"]}]
    (tmp_path / "o").mkdir()
    out, real_in = io.StringIO(), sys.stdin
    sys.stdin, sys.stdout = io.StringIO("".join(json.dumps(s) + "\n" for s in steps)), out
    try:
        assert main(["trace-run", "--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(tmp_path / "o"),
                     "--max-tokens", "128"]) == 0
    finally:
        sys.stdin, sys.stdout = real_in, real
    assert out.getvalue().split() == ["done", "0", "done", "1"] and not (tmp_path / "o" / "0.f32").exists()
    data = (tmp_path / "o" / "1.f32").read_bytes()
    got = torch.tensor(struct.unpack(f"<{len(data) // 4}f", data)).view(3, cfg.vocab_size)
    want = torch.stack([b.ref(prompt)[-1], b.ref([1, 2])[1], b.ref([1, 2])[0]])
    assert worst_row(got, want) < TOL[F32]
    assert math.isfinite(float(got.sum()))
