"""Nugosun on the GPU against the plain restatement in ``oracle/nugosun.py``: every mechanism alone, then the model
through its ragged batches, its decode engine, the serving engine and the command line, in 32-bit (tight) and bf16."""
import io
import json
import struct
import sys
from dataclasses import replace

import pytest
import torch
from oracle import nugosun as O
from torch.nn.functional import silu

from rmlx_b200.config import (ChosenFfSpec, ChunkedAttentionSpec, GlaSpec, LatentAttentionSpec, NugosunConfig, PairSpec,
                              RotarySpec, SamplerConfig, SchedulerConfig, StateSpaceSpec, SwigluFfSpec, TwinNormLayerSpec)
from rmlx_b200.models import nugosun as M
from rmlx_b200.models.ragged import Entry, RaggedBatch, query_tiles
from rmlx_b200.models.ragged_model import Buffers, StepContext
from rmlx_b200.models.twin_norm_decode import TwinNormDecode
from rmlx_b200.ops import parallel_block as P
from rmlx_b200.ops import routed as R
from rmlx_b200.ops import scan as S
from rmlx_b200.ops import twin_norm as TN
from rmlx_b200.serve.engine import ServingEngine

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32
pad8 = P.pad8
YARN = {"factor": 5.0, "original": 64.0, "fast": 6.0, "slow": 0.7}


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


def one_layer(mixer, mlp=None, width=40, eps=1e-5, seed=0, change=None):
    """(config, checkpoint tensors in fp32) of a model of one layer; ``change`` edits the tensors."""
    cfg = NugosunConfig(16, width, [TwinNormLayerSpec(mixer, mlp)], eps).validate()
    t = {k: v.float() for k, v in M.random_tensors(cfg, seed).items()}
    if change is not None:
        change(t)
    return cfg, t


def mix_of(t, dtype=torch.float64):
    return {k[7:]: v.to(dtype) for k, v in t.items() if k.startswith("l0.mix.")}


# ------------------------------------------------------------------ chunked attention
class ChunkedHeads:
    """q, k and v of several sequences in pages; attention inside chunks with a soft cap by the oracle."""

    def __init__(self, dev, lens, hq, hkv, dk, dv, dtype=BF, seed=0, cap=12.0, sharp=1.0):
        r = rand(seed)
        self.dev, self.lens, self.hq, self.hkv, self.dk, self.dv, self.dtype = dev, lens, hq, hkv, dk, dv, dtype
        self.q, self.k = [r(n, hq, dk).to(dtype) for n in lens], [r(n, hkv, dk).to(dtype) for n in lens]
        self.v, self.scale, self.cap = [r(n, hkv, dv).to(dtype) for n in lens], sharp * dk ** -0.5, cap

    def build(self):
        table, count = shuffled_pages(self.lens)
        kc = torch.zeros(count, self.hkv, 16, pad8(self.dk), dtype=self.dtype)
        vc = torch.zeros(count, self.hkv, 16, pad8(self.dv), dtype=self.dtype)
        for s, n in enumerate(self.lens):
            for t in range(n):
                kc[table[s, t // 16], :, t % 16, :self.dk] = self.k[s][t]
                vc[table[s, t // 16], :, t % 16, :self.dv] = self.v[s][t]
        return kc.to(self.dev), vc.to(self.dev), table.to(self.dev)

    def want(self, rows, chunk):
        outs = {}
        for s in {s for s, _ in rows}:
            q, k, v = (x[s].double().permute(1, 0, 2) for x in (self.q, self.k, self.v))
            k, v = k.repeat_interleave(self.hq // self.hkv, 0), v.repeat_interleave(self.hq // self.hkv, 0)
            z = q @ k.transpose(1, 2) * self.scale
            z = self.cap * torch.tanh(z / self.cap) if self.cap else z
            outs[s] = O.softmax_attention(z, O.same_chunk(self.lens[s], chunk) if chunk else O.visible(self.lens[s]), v)
        return torch.stack([outs[s][:, t] for s, t in rows])

    def every_kernel(self, rows, starts, chunk):
        """The rows (sequences' tails from ``starts``) through every attention kernel that takes them."""
        kc, vc, table = self.build()
        q = torch.zeros(len(rows), self.hq, pad8(self.dk), dtype=self.dtype)
        for i, (s, t) in enumerate(rows):
            q[i, :, :self.dk] = self.q[s][t]
        q, mods = q.to(self.dev), P.ScoreMods(self.scale, self.cap)
        pos, seq = i32([t for _, t in rows], self.dev), i32([s for s, _ in rows], self.dev)
        new = lambda: torch.full((len(rows), self.hq, pad8(self.dv)), 5.0, dtype=self.dtype, device=self.dev)   # noqa: E731
        outs = {"any": P.attention_any(q, kc, vc, table, pos, seq, mods, new(), chunk=chunk)}
        if self.dtype == BF and P.prefill_scored_supported(pad8(self.dk), pad8(self.dv)):
            lens = [n - lo for n, lo in zip(self.lens, starts)]
            firsts = [sum(lens[:i]) for i in range(len(lens))]
            for lanes in (1, 2):
                tiles = i32(query_tiles(firsts, lens, starts, list(range(len(lens))), 128 * lanes), self.dev)
                outs[f"prompt{lanes}"] = P.flash_prefill_scored(q, kc, vc, table, tiles, mods, new(), lanes=lanes, chunk=chunk)
            for splits in (1, 3):
                scr = P.ScoredDecodeScratch(len(rows), self.hq, self.hkv, pad8(self.dv), splits, self.dev)
                outs[f"decode{splits}"] = P.flash_decode_scored(kc, vc, table, pos, mods, new(), scr, self.hq, self.dk,
                                                                self.dv, q=q, table_rows=seq, chunk=chunk)
        return {n: o[..., :self.dv] for n, o in outs.items()}


@pytest.mark.parametrize("shape,cap", [((4, 2, 32, 40), 12.0), ((6, 6, 72, 16), 0.0), ((8, 1, 128, 128), 3.0),
                                       ((2, 1, 136, 24), 5.0)], ids=str)
@pytest.mark.parametrize("dtype,tol", [(F32, 2e-6), (BF, 7e-3)])
@pytest.mark.parametrize("chunk", [0, 1, 16, 37, 64, 130, 1000])
def test_chunked_attention(dev, shape, cap, dtype, tol, chunk):
    h = ChunkedHeads(dev, [3, 18, 300], *shape, dtype=dtype, cap=cap)
    starts = [0, 1, 45]
    rows = [(s, t) for s, lo in enumerate(starts) for t in range(lo, h.lens[s])]
    want = h.want(rows, chunk)
    for name, got in h.every_kernel(rows, starts, chunk).items():
        assert rel(got, want) < tol, name


def test_chunk_edges_stand_out(dev):
    """A key that is its chunk's first carries most of one query's weight; the token before it, as strong, none."""
    for chunk in (15, 16, 17, 48, 64, 100):
        h = ChunkedHeads(dev, [260], 2, 1, 64, 32, seed=7, cap=0.0)
        picks = [t for t in (150, 160, 191, 200, 255) if t % chunk > 2]
        for t in picks:
            for key in (t - t % chunk, t - t % chunk - 1):
                h.k[0][key] = (h.q[0][t].float()[0] * 3).to(BF)
        rows = [(0, t) for t in range(100, 260)]
        want = h.want(rows, chunk)
        at = [t - 100 for t in picks]
        assert rel(h.want(rows, chunk + 1)[at], want[at]) > 0.2          # on the CPU: another size is far off
        for name, got in h.every_kernel(rows, [100], chunk).items():
            assert rel(got, want) < 8e-3, (name, chunk)
            for t in at:
                assert rel(got[t], want[t]) < 2e-2, (name, chunk, t)


def turned(raw, heads, spec, eps, pos):
    """A head's rows after rotation at ``pos`` and norm, by the oracle (rows of a longer sequence)."""
    x = torch.zeros(heads, pos + 1, raw.shape[-1], dtype=torch.float64)
    x[:, pos] = raw
    return O.rms_norm(O.rotate_halves(x, spec), eps)[:, pos]


ROTARY = [{"base": 500.0, "dims": 20}, {"base": 1e4, "dims": 24, "scaling": YARN}, {"base": 1e4, "dims": 0},
          {"base": 7e4, "dims": 6, "scaling": {"factor": 1.0, "original": 8.0, "fast": 2.0, "slow": 1.9}}]


@pytest.mark.parametrize("dtype,tol", [(F32, 2e-6), (BF, 5e-3)])
@pytest.mark.parametrize("hq,hkv,dk,dv", [(3, 1, 24, 10), (6, 3, 72, 40), (2, 2, 300, 8)])
@pytest.mark.parametrize("rot", ROTARY, ids=lambda r: f"{r['dims']}{'y' if 'scaling' in r else ''}")
def test_bias_rotation_norm_append(dev, dtype, tol, hq, hkv, dk, dv, rot):
    r, eps = rand(1), 1e-3
    nq, nk, nv = hq * dk, hkv * dk, hkv * dv
    pos, seq = list(range(14, 31)) + list(range(20)) + [90], [0] * 17 + [1] * 20 + [2]
    t = len(pos)
    raw, bias = r(t, pad8(nq + nk + nv)).to(dtype), 0.5 * r(nq + nk + nv)
    f, grow = TN.rotary_frequencies(rot["base"], rot["dims"], rot.get("scaling"))
    kc = torch.zeros(12, hkv, 16, pad8(dk), dtype=dtype, device=dev)
    vc = torch.zeros(12, hkv, 16, pad8(dv), dtype=dtype, device=dev)
    table = i32([[4, 2, 8, 0, 0, 0], [7, 1, 3, 0, 0, 0], [0, 0, 0, 0, 0, 9]], dev)
    q = torch.full((t, hq, pad8(dk)), 5.0, dtype=dtype, device=dev)
    TN.rotary_norm_append(raw.to(dev), bias.to(dev), f.float().to(dev), grow, eps, q, kc, vc, table, i32(pos, dev),
                          i32(seq, dev), hq, dk, dv)
    d = raw.double()[:, :nq + nk + nv] + bias.double()
    for i in (0, 3, 16, 17, 36, t - 1):
        assert rel(q[i, :, :dk], turned(d[i, :nq].view(hq, dk), hq, rot, eps, pos[i])) < tol
        page, off = int(table[seq[i], pos[i] // 16]), pos[i] % 16
        assert rel(kc[page, :, off, :dk], turned(d[i, nq:nq + nk].view(hkv, dk), hkv, rot, eps, pos[i])) < tol
        assert rel(vc[page, :, off, :dv], d[i, nq + nk:].view(hkv, dv)) < tol
    assert not q[..., dk:].any() and not kc[..., dk:].any() and not vc[..., dv:].any() and not kc[[0, 5, 6, 10]].any()


@pytest.mark.parametrize("shape", [(4, 2, 32, 40), (2, 2, 20, 72), (40, 2, 64, 64), (16, 1, 128, 128)], ids=str)
@pytest.mark.parametrize("chunk,rot", [(0, ROTARY[0]), (17, {"base": 1e4, "dims": 18, "scaling": YARN}), (64, ROTARY[2])])
def test_fused_bias_rotation_norm_append_attention(dev, shape, chunk, rot):
    """The decode form: one launch on the projection's fp32 rows."""
    hq, hkv, dk, dv = shape
    r, lens = rand(3), [1, 16, 17, 200]
    h = ChunkedHeads(dev, lens, *shape, seed=2)
    nq, nk, nv = hq * dk, hkv * dk, hkv * dv
    raw, bias = r(4, nq + nk + nv + 5), 0.4 * r(nq + nk + nv)
    d = raw[:, :nq + nk + nv].double() + bias.double()
    for s, n in enumerate(lens):                          # the oracle's view of the new token
        h.q[s][n - 1] = turned(d[s, :nq].view(hq, dk), hq, rot, 1e-5, n - 1).to(BF)
        h.k[s][n - 1] = turned(d[s, nq:nq + nk].view(hkv, dk), hkv, rot, 1e-5, n - 1).to(BF)
        h.v[s][n - 1] = d[s, nq + nk:].view(hkv, dv).to(BF)
    want_k, want_v, table = h.build()
    kc, vc = want_k.clone(), want_v.clone()
    for s, n in enumerate(lens):                          # the slot of the new token starts dirty
        kc[table[s, (n - 1) // 16], :, (n - 1) % 16, :dk] = 9.0
        vc[table[s, (n - 1) // 16], :, (n - 1) % 16, :dv] = -9.0
    f, grow = TN.rotary_frequencies(rot["base"], rot["dims"], rot.get("scaling"))
    for splits in (1, 5):
        out = torch.zeros(4, hq, pad8(dv), dtype=BF, device=dev)
        scr = P.ScoredDecodeScratch(4, hq, hkv, pad8(dv), splits, dev)
        P.flash_decode_scored(kc, vc, table, i32([n - 1 for n in lens], dev), P.ScoreMods(h.scale, h.cap), out, scr, hq, dk, dv,
                              raw=raw.to(dev), eps=1e-5, chunk=chunk, head_norm=True, bias=bias.to(dev),
                              inv_freq=f.float().to(dev), grow=grow)
        assert rel(out[..., :dv], h.want([(s, n - 1) for s, n in enumerate(lens)], chunk)) < 7e-3
        assert rel(kc, want_k) < 3e-3 and rel(vc, want_v) < 3e-3


# ------------------------------------------------------------------ mixers over a cache of their own
class MixerCase:
    """A model of one layer without feed-forward; its mixer over whole sequences by the oracle."""

    def __init__(self, dev, mixer, dtype, seed=0, width=40, change=None):
        self.dev, self.dtype, self.width = dev, dtype, width
        self.cfg, t = one_layer(mixer, None, width, seed=seed, change=change)
        self.t = {k: v if v.dim() == 1 else v.to(dtype).float() for k, v in t.items()}
        self.model = M.NugosunModel(M.build_weights(self.cfg, self.t, dev, dtype))
        self.mw, self.w = self.model.w.layers[0].mix, mix_of(self.t)
        self.cache = self.model.new_cache(80, max_seqs=6)

    def rows(self, h):
        x = torch.zeros(len(h), pad8(self.width), dtype=self.dtype, device=self.dev)
        x[:, :self.width] = h.to(self.dev)
        return x

    def add(self, terms):
        """Sum of the terms' projections, fp32 [T, width]."""
        x = torch.zeros(terms[0][0].shape[0], pad8(self.width), device=self.dev)
        self.model.add_terms(x, terms, StepContext(len(x), None, None, None, None, None, None, None))
        return x[:, :self.width]

    def run(self, forward, hs, cuts):
        """The sequences' rows in portions (all that are left to cut share a batch), continued on the cache."""
        ids = list(range(len(hs)))
        for i in ids:
            self.cache.add_sequence(i)
        got, at = [[] for _ in hs], [0] * len(hs)
        for cut in cuts:
            live = [i for i in ids if cut[i]]
            for i in live:
                self.cache.reserve(i, cut[i])
            b = RaggedBatch.plan([Entry(i, [0] * cut[i]) for i in live], self.cache, 1, self.model._absorb).upload(self.dev)
            c = StepContext(b.num_tokens, Buffers(256, self.dev), self.cache, self.cache.block_table, b.positions, b.token_seq,
                            b.token_seq, b.runs, b)
            out = self.add(forward(0, self.mw, self.rows(torch.cat([hs[i][at[i]:at[i] + cut[i]] for i in live])), c))
            lo = 0
            for i in live:
                got[i].append(out[lo:lo + cut[i]].cpu())
                lo += cut[i]
                at[i] += cut[i]
                self.cache.commit(i, cut[i])
        assert at == [len(h) for h in hs]
        return [torch.cat(g) for g in got]


CUTS = ([1, 1, 2, 3], [0, 2, 17, 16], [0, 1, 1, 1], [0, 1, 30, 13])
LENS = [1, 5, 50, 33]
GLA = [GlaSpec(3, 7, 12, 16.0, 5), GlaSpec(2, 16, 33, 4.0, 16), GlaSpec(1, 64, 64, 1.0, 3), GlaSpec(2, 100, 20, 9.0, 24),
       GlaSpec(1, 200, 264, 16.0, 16)]
SSD = [StateSpaceSpec(4, 12, 7, 2, 3, 3), StateSpaceSpec(6, 16, 33, 3, 4, 1), StateSpaceSpec(2, 64, 64, 1, 1, 2),
       StateSpaceSpec(2, 40, 100, 2, 2, 1), StateSpaceSpec(1, 24, 200, 1, 7, 4)]
CHUNKED = ChunkedAttentionSpec(4, 2, 32, 24, 0.3, RotarySpec(1e3, 12, YARN), 9.0, 13)
GLA_ID = lambda m: f"{m.heads}-{m.dim}-{m.vdim}"                          # noqa: E731
SSD_ID = lambda m: f"{m.heads}-{m.vdim}-{m.state}-{m.groups}-{m.conv}"    # noqa: E731


def portions(dtype, tol, case, forward, want):
    hs = [rand(40 + i)(n, case.width).to(dtype) for i, n in enumerate(LENS)]
    got = case.run(forward, hs, CUTS)
    for g, h in zip(got, hs):
        assert rel(g, want(h.double())) < tol


@pytest.mark.parametrize("spec", GLA, ids=GLA_ID)
@pytest.mark.parametrize("dtype,tol", [(F32, 5e-6), (BF, 1.5e-2)])
def test_gated_linear_attention_in_portions(dev, spec, dtype, tol):
    c = MixerCase(dev, spec, dtype)
    portions(dtype, tol, c, c.model.linear_attention, lambda h: O.gated_linear_attention(c.w, spec.to_json(), 1e-5, h))


@pytest.mark.parametrize("spec", SSD, ids=SSD_ID)
@pytest.mark.parametrize("dtype,tol", [(F32, 1e-5), (BF, 2e-2)])
def test_state_space_beside_attention_in_portions(dev, spec, dtype, tol):
    """Both halves of a pair with their factors; portions cut inside the convolution's reach."""
    pair = PairSpec(CHUNKED, spec, 0.7, 1.6)
    c = MixerCase(dev, pair, dtype)
    portions(dtype, tol, c, c.model.pair, lambda h: O.side_by_side(c.w, pair.to_json(), 1e-5, h))
    right = {k[6:]: v for k, v in c.w.items() if k.startswith("right.")}
    h = rand(9)(20, 40).double()
    want = O.side_by_side(c.w, pair.to_json(), 1e-5, h)
    assert rel(0.7 * O.chunked_attention({k[5:]: v for k, v in c.w.items() if k.startswith("left.")}, pair.left.to_json(), 1e-5, h)
               + 1.6 * O.state_space(right, spec.to_json(), 1e-5, h), want) < 1e-12


LATENT = [LatentAttentionSpec(3, 24, 16, 40, 72, 0.2, 100.0, q_rank=20), LatentAttentionSpec(5, 12, 6, 10, 21, 0.3, 500.0, 4, q_rank=33),
          LatentAttentionSpec(2, 128, 64, 128, 128, 0.07, 1e4, q_rank=64)]


@pytest.mark.parametrize("spec", LATENT, ids=lambda s: f"{s.heads}-{s.dim}-{s.rot_dim}-{s.vdim}-{s.kv_rank}-{s.q_rank}")
@pytest.mark.parametrize("dtype,tol", [(F32, 5e-6), (BF, 3e-2)])
def test_latent_attention_with_a_query_latent_in_portions(dev, spec, dtype, tol):
    c = MixerCase(dev, spec, dtype)
    m = spec.to_json()
    portions(dtype, tol, c, c.model.latent_attention,
             lambda h: O.latent_attention(c.w, m, 1e-5, h, O.latent_rows(c.w, m, 1e-5, h)))


def shared_rows_model(dev, dtype):
    """Two latent layers, the second on the first one's rows with other heads, sizes and query rank."""
    a = LatentAttentionSpec(4, 24, 16, 24, 40, 0.4, 300.0, q_rank=24)
    b = replace(a, heads=3, dim=40, vdim=16, scale=0.5, q_rank=52, kv_from=0)
    cfg = NugosunConfig(50, 64, [TwinNormLayerSpec(a, SwigluFfSpec(40)), TwinNormLayerSpec(b, None)], 1e-4).validate()
    t = M.random_tensors(cfg, 6)
    return cfg, t, M.NugosunModel(M.build_weights(cfg, t, dev, dtype))


@pytest.mark.parametrize("dtype,tol", [(F32, 2e-5), (BF, 6e-2)])
def test_rows_shared_between_layers(dev, dtype, tol):
    cfg, t, model = shared_rows_model(dev, dtype)
    assert model.w.layers[1].mix.c_norm is None and model.new_cache(4).k[1] is None
    toks, w = torch.randint(0, 50, (70,), generator=torch.Generator().manual_seed(1)).tolist(), {k: v.double() for k, v in t.items()}
    want = O.forward(cfg.to_json(), w, toks)
    own = cfg.to_json()                                   # on the CPU: rows of its own would be far off
    own["layers"][1]["mixer"].pop("kv_from")
    w2 = {**w, **{k.replace("l0.mix.dkv", "l1.mix.dkv"): v.flip(0) for k, v in w.items() if "l0.mix.dkv" in k}}
    assert worst_row(O.forward(own, w2, toks), want) > 0.1
    cache = model.new_cache(12, max_seqs=2)
    cache.add_sequence(0)
    got = [model.forward_batch([Entry(0, toks[:37], range(37))], cache)]
    got += [model.forward_batch([Entry(0, toks[37:39], range(2))], cache)]
    got += [model.forward_batch([Entry(0, [x], [0])], cache) for x in toks[39:45]]
    got.append(model.forward_batch([Entry(0, toks[45:], range(25))], cache))
    assert worst_row(torch.cat(got), want) < tol


def test_states_decay_exactly_over_a_long_past(dev):
    """One strong key at the start is read back hundreds of tokens later through slow decays: a lost or repeated decay
    step shows."""
    h, n, d, t = 2, 24, 40, 600
    r = rand(9)
    q, k, v = 0.01 * r(t, h * n), 0.01 * r(t, h * n), r(t, h * d)
    k[3], q[t - 1] = 3.0, 1.0
    z, bias = 2 + 0.3 * r(t, h * n), 0.2 * r(h * n)
    hf = lambda x, c=h: O.heads_first(x.double(), c)                      # noqa: E731
    decay = torch.exp(torch.nn.functional.logsigmoid((z + bias).double()) / 30.0)
    want = O.heads_last(O.outer_recurrence(hf(q) * 0.3, hf(k), hf(v), hf(decay)))
    lost = decay.clone()
    lost[300] = 1.0
    assert rel(O.heads_last(O.outer_recurrence(hf(q) * 0.3, hf(k), hf(v), hf(lost)))[-1], want[-1]) > 1e-3
    state = torch.zeros(2, h, n, d, device=dev)
    o = torch.zeros(t, h * d, device=dev)
    wide = torch.zeros(t, 2 * h * n + h * d, device=dev)                  # one row stride for q, k and v
    qd, kd, vd = wide[:, :h * n], wide[:, h * n:2 * h * n], wide[:, 2 * h * n:]
    qd.copy_(q), kd.copy_(k), vd.copy_(v)
    S.gla_scan(qd, kd, vd, z.to(dev), bias.to(dev), 30.0, 0.3, state, o, torch.empty(t * h * S.record(n, d), device=dev),
               runs=i32([[0, t, 0, 0]], dev))
    assert rel(o[-1], want[-1]) < 2e-5 and rel(o, want) < 2e-5 and not state[1].any()

    # state-space heads: a slow head keeps the first token's input, the convolution is a plain copy
    H, G, N, D = 2, 1, 8, 4
    ch = H * D + 2 * G * N
    raw = torch.zeros(t, ch + H)
    raw[:, :ch] = 0.01 * r(t, ch)
    raw[0, :H * D], raw[0, H * D:H * D + N], raw[t - 1, H * D + N:ch] = 4.0, 4.0, 4.0
    raw[:, ch:] = -4 + 0.2 * r(t, H)
    conv = torch.zeros(2, ch)
    conv[1] = 1.0
    a_log, skip = torch.tensor([-3.0, -2.0]), torch.tensor([0.0, 0.1])

    def plain(drop=None):
        s = silu(raw[:, :ch].double())
        x, b, c = torch.split(s, [H * D, N, N], -1)
        dt = torch.nn.functional.softplus(raw[:, ch:].double())
        a = torch.exp(-torch.exp(a_log.double()) * dt)
        if drop is not None:
            a[drop] = 1.0
        b, c = (O.heads_first(y, G).repeat_interleave(H, 0) for y in (b, c))
        y = O.outer_recurrence(c, b * dt.T[:, :, None], O.heads_first(x, H), a.T[:, :, None].expand(-1, -1, N))
        return O.heads_last(y + skip.double()[:, None, None] * O.heads_first(x, H))

    want = plain()
    assert rel(plain(300)[-1], want[-1]) > 2e-4
    pool = torch.zeros(3, H * N * D + ch, device=dev)
    st, carried = pool[:, :H * N * D].unflatten(1, (H, N, D)), pool[:, H * N * D:].unflatten(1, (1, ch))
    o = torch.zeros(t, H * D, device=dev)
    S.ssd_scan(raw.to(dev), 0, ch, conv.to(dev), torch.zeros(ch, device=dev), carried, torch.zeros(H, device=dev), a_log.to(dev),
               skip.to(dev), G, st, o, torch.empty(t * H * S.record(N, D, True, H // G), device=dev),
               i32([2] * t, dev), runs=i32([[0, t, 2, 0]], dev))
    assert rel(o[-1], want[-1]) < 2e-5 and rel(o, want) < 2e-5 and not pool[:2].any()
    assert torch.equal(carried[2, 0].cpu(), raw[-1, :ch])


def test_convolution_inputs_cross_portions(dev):
    """Taps that only look back: what a portion reads from before its start comes from the carried inputs."""
    spec = StateSpaceSpec(2, 8, 8, 1, 5, 1)
    pair = PairSpec(replace(CHUNKED, chunk=0), spec, 0.0, 1.0)

    def back_only(t):
        t["l0.mix.right.conv"][:, 1:] = 0.0
        t["l0.mix.right.conv"][:, 0] = 2.0

    c = MixerCase(dev, pair, F32, change=back_only)
    h = rand(3)(23, 40)
    want = O.side_by_side(c.w, pair.to_json(), 1e-5, h.double())
    w = dict(c.w)
    w["right.conv"] = torch.roll(w["right.conv"], 1, 1)                   # one token off is far off
    assert rel(O.side_by_side(w, pair.to_json(), 1e-5, h.double()), want) > 0.3
    got = c.run(c.model.pair, [h], [[2], [1], [1], [3], [2], [9], [1], [4]])
    assert rel(got[0], want) < 1e-5


@pytest.mark.parametrize("groups,size", [(1, 20), (3, 24), (2, 130), (4, 512), (1, 1500)])
@pytest.mark.parametrize("dtype,tol", [(F32, 1e-6), (BF, 4e-3)])
def test_grouped_gated_norm(dev, groups, size, dtype, tol):
    r, n = rand(size), groups * size
    o, z, w = r(9, n), (2 * r(9, n)).to(dtype), 1 + 0.2 * r(n)
    out = torch.full((9, n + 3), 7.0, dtype=dtype, device=dev)
    S.gated_norm(o.to(dev), z.to(dev), w.to(dev), 1e-2, groups, out, True)
    want = O.grouped_gated_norm(o.double(), z.double(), groups, 1e-2, w.double())
    assert rel(out[:, :n], want) < tol and (out[:, n:] == 7).all()
    S.gated_norm(o.to(dev), z.to(dev), w.to(dev), 1e-2, groups, out, False)
    want = O.rms_norm(o.double().view(9, groups, size), 1e-2).view(9, n) * w.double() * silu(z.double())
    assert rel(out[:, :n], want) < tol


# ------------------------------------------------------------------ norms, feed-forward, routing
@pytest.mark.parametrize("width", [20, 104, 2100, 9000])
@pytest.mark.parametrize("dtype,tol", [(F32, 2e-6), (BF, 4e-3)])
def test_two_norms_of_one_row(dev, width, dtype, tol):
    r, t, ldx = rand(width), 7, pad8(width)
    vec = lambda: torch.nn.functional.pad(1 + 0.3 * r(width), (0, ldx - width))             # noqa: E731
    x = torch.nn.functional.pad(3 * r(t, width), (0, ldx - width)).to(dev)
    w1, w2 = vec(), vec()
    new = lambda: torch.full((t, ldx), 9.0, dtype=dtype, device=dev)      # noqa: E731
    h1, h2, before = new(), new(), x.clone()
    TN.twin_norm(x, w1.to(dev), h1, w2.to(dev), h2, 1e-2, width)
    for h, w in ((h1, w1), (h2, w2)):
        assert rel(h[:, :width], O.rms_norm(x[:, :width].double().cpu(), 1e-2, w[:width].double())) < tol and not h[:, width:].any()
    assert torch.equal(x, before)
    # with experts' rows: slots in any order, more than four of them, one token's all alike
    for top in (1, 3, 6):
        y = torch.zeros(t * top, ldx + 8)
        y[:, :width] = r(t * top, width)
        y[:, width:] = 50.0                               # past the width: nobody's
        order = torch.randperm(t * top, generator=torch.Generator().manual_seed(top)).int().view(t, top)
        wt = torch.rand(t, top, generator=torch.Generator().manual_seed(top))
        i = lambda *s: torch.zeros(*s, dtype=torch.int32, device=dev)     # noqa: E731
        rt = R.Routing(i(t, top), wt.to(dev), None, i(1), i(2), order.to(dev))
        yd = y.to(dtype)
        want = before[:, :width].double().cpu() + (wt.double()[:, :, None] * yd[:, :width].double()[order.long()]).sum(1)
        x.copy_(before)
        TN.twin_norm(x, w1.to(dev), h1, None, None, 1e-2, width, (yd.to(dev), rt))
        assert rel(x[:, :width], want) < 1e-6 and not x[:, width:].any()
        assert rel(h1[:, :width], O.rms_norm(want, 1e-2, w1[:width].double())) < tol
        x.copy_(before)
        TN.twin_norm(x, None, None, None, None, 1e-2, width, (yd.to(dev), rt))
        assert rel(x[:, :width], want) < 1e-6


@pytest.mark.parametrize("e,top", [(1, 1), (5, 1), (6, 6), (40, 8), (70, 3), (300, 12)])
def test_routing_by_biased_logits(dev, e, top):
    r, t = rand(e), 53
    z, bias = 2 * r(t, e), 0.7 * r(e)
    i = lambda *s: torch.zeros(*s, dtype=torch.int32, device=dev)         # noqa: E731
    rt = R.Routing(i(t, top), torch.zeros(t, top, device=dev), None, i(e), i(e + 1), i(t, top))
    R.route_chosen(z.to(dev), bias.to(dev), rt)
    idx, wt = O.route(torch.eye(e, dtype=torch.float64), bias.double(), top, z.double())
    got, order = rt.idx.cpu().long().sort(1)
    want, back = idx.sort(1)
    assert torch.equal(got, want)
    assert rel(rt.weights.cpu().gather(1, order), wt.gather(1, back)) < 1e-6
    assert torch.allclose(rt.weights.sum(1).cpu(), torch.ones(t), atol=1e-5)
    count = torch.bincount(got.reshape(-1), minlength=e)
    assert torch.equal(rt.offsets.cpu().long(), torch.cat([torch.zeros(1, dtype=torch.long), count.cumsum(0)]))


@pytest.mark.parametrize("dtype,tol", [(F32, 5e-6), (BF, 1e-2)])
@pytest.mark.parametrize("t,e,top", [(1, 3, 2), (70, 6, 3), (300, 4, 1), (9, 6, 6)])
def test_routed_feed_forward(dev, dtype, tol, t, e, top):
    cfg, tensors = one_layer(GlaSpec(1, 8, 8, 2.0), ChosenFfSpec(e, top, 40), 44, 1e-4, 7)
    tensors = {k: v.to(dtype).float() for k, v in tensors.items()}
    model = M.NugosunModel(M.build_weights(cfg, tensors, dev, dtype))
    f, r = model.w.layers[0].mlp, rand(t)
    h = torch.zeros(t, 48, dtype=dtype, device=dev)
    h[:, :44] = r(t, 44).to(dev)
    x = torch.zeros(t, 48, device=dev)
    c = StepContext(t, Buffers(max(t, 8), dev), None, None, None, None, None, None)
    rt = model.routing(f, c)
    R.route_chosen(model.router_logits(f, h, c), f.correction, rt)
    TN.twin_norm(x, None, None, None, None, 1e-4, 44, (model.expert_rows(f, h, rt, c), rt))
    mlp = {k[7:]: v.double() for k, v in tensors.items() if k.startswith("l0.mlp.")}
    assert rel(x[:, :44], O.expert_mix(mlp, cfg.layers[0].mlp.to_json(), h[:, :44].double().cpu())) < tol


# ------------------------------------------------------------------ decode kernels
@pytest.mark.parametrize("b", [1, 3, 6])
@pytest.mark.parametrize("d", [100, 700])
def test_decode_projections_of_two_norms(dev, b, d):
    r, k = rand(b), pad8(d)
    pad = lambda v: torch.nn.functional.pad(v, (0, k - v.shape[-1]))      # noqa: E731
    x, w1, w2 = pad(3 * r(b, d)), pad(1 + 0.2 * r(d)), pad(1 + 0.4 * r(d))
    n1, n2 = (O.rms_norm(x[:, :d].double(), 1e-4, w[:d].double()) for w in (w1, w2))
    w, gu = pad(r(1075, d) / 10).to(BF), pad(r(2 * 360, d) / 10).to(BF)
    dv = lambda *v: [y.to(dev) for y in v]                                # noqa: E731
    xd, w1d, w2d, wd, gud = dv(x, w1, w2, w, gu)
    want, gate = n1 @ w[:, :d].double().T, silu(n2 @ gu[:360, :d].double().T) * (n2 @ gu[360:, :d].double().T)
    out, act = torch.empty(b, 1075, device=dev), torch.empty(b, 360, dtype=BF, device=dev)
    TN.twin_in(xd, w1d, 1e-4, d, wd, out)
    assert rel(out, want) < 3e-6
    out.zero_()
    TN.twin_in(xd, w1d, 1e-4, d, wd, out, w2d, gud, act)
    assert rel(out, want) < 3e-6 and rel(act, gate) < 5e-3
    e, top, ff = 9, 4, 64
    router, bias = pad(r(e, d) / 3).to(BF), 0.5 * r(e)
    i = lambda *s: torch.zeros(*s, dtype=torch.int32, device=dev)         # noqa: E731
    rt = R.Routing(i(b, top), torch.zeros(b, top, device=dev), None, i(e), i(e + 1), i(b, top))
    z, h2, ticket = torch.empty(b, e, device=dev), torch.full((b, k), 7.0, device=dev), i(1)
    for _ in range(2):                                    # the ticket is left clean
        out.zero_()
        TN.twin_in_router(xd, w1d, 1e-4, d, wd, out, w2d, router.to(dev), bias.to(dev), z, h2, ticket, rt)
    assert rel(out, want) < 3e-6 and rel(h2[:, :d], n2) < 2e-6 and not h2[:, d:].any() and int(ticket) == 0
    ew = {"router": router[:, :d].double(), "router.b": bias.double()}
    for j in range(e):
        ew.update({f"e{j}.gate": (r(ff, d) / d ** 0.5).to(BF), f"e{j}.up": (r(ff, d) / d ** 0.5).to(BF),
                   f"e{j}.down": (r(d, ff) / 8).to(BF)})
    stack = lambda n: torch.stack([ew[f"e{j}.{n}"] for j in range(e)])    # noqa: E731
    gus = pad(torch.cat([stack("gate"), stack("up")], 1).float()).to(BF).to(dev)
    downs = torch.zeros(e, (d + 127) // 128 * 128, ff, dtype=BF, device=dev)
    downs[:, :d] = stack("down").to(dev)
    acte = torch.zeros(b * top, ff, dtype=BF, device=dev)
    R.postnorm_expert(h2, gus, 0.0, rt, acte)
    y, ones = xd.clone(), torch.ones(max(b, 8), device=dev)
    R.expert_out(acte, downs, replace(rt, identity=ones), y, y)           # into the residual, in place
    mix = O.expert_mix({n: v.double() for n, v in ew.items()}, ChosenFfSpec(e, top, ff).to_json(), n2)
    assert rel(y[:, :d] - xd[:, :d], mix) < 8e-3 and not y[:, d:].any()


def decode_against(case, forward, want_of, b, tol):
    """Six tokens of ``b`` rows in shuffled slots, one at a time."""
    slots = torch.randperm(6, generator=torch.Generator().manual_seed(1))[:b].int().to(case.dev)
    h = rand(b)(b, 6, case.width)
    want = [want_of(h[i].double()) for i in range(b)]
    for t in range(6):
        x = torch.zeros(b, pad8(case.width), device=case.dev)
        x[:, :case.width] = h[:, t].to(case.dev)
        raw = torch.empty(b, case.mw.w_in.n, device=case.dev)
        # no norm here: the rows are what the mixer reads
        raw.copy_(x.double() @ case.mw.w_in.w.double().T)
        got = case.add(forward(raw, slots))
        assert rel(got, torch.stack([w[t] for w in want])) < tol, t


@pytest.mark.parametrize("spec", GLA + [GlaSpec(2, 128, 256, 16.0, 16), GlaSpec(2, 32, 300, 5.0, 8)], ids=GLA_ID)
@pytest.mark.parametrize("b", [1, 3])
def test_gated_linear_attention_decode_step(dev, spec, b):
    c = MixerCase(dev, spec, BF)
    state = c.cache.layer_state(0, "gla")

    def step(raw, slots):
        a = torch.zeros(b, c.mw.v_p, dtype=BF, device=dev)
        S.gla_decode(raw, c.mw.at, c.mw.w_a2, c.mw.bias, spec.tau, spec.dim ** -0.5, c.mw.norm, 1e-5, slots, state, a)
        return [(a, c.mw.w_o, c.model.w.ones)]

    decode_against(c, step, lambda h: O.gated_linear_attention(c.w, spec.to_json(), 1e-5, h), b, 6e-3)
    assert int((c.cache.state.abs().sum(1) > 0).sum()) == b               # other slots are untouched


@pytest.mark.parametrize("spec", SSD + [StateSpaceSpec(4, 64, 128, 1, 4, 1)], ids=SSD_ID)
@pytest.mark.parametrize("b", [1, 3])
def test_state_space_decode_step(dev, spec, b):
    c = MixerCase(dev, PairSpec(CHUNKED, spec, 0.0, 1.3), BF)
    w, r = c.mw.right, {k[6:]: v for k, v in c.w.items() if k.startswith("right.")}
    state = c.cache.layer_state(0, "ssd")
    carried = c.cache.layer_state(0, "conv") if spec.conv > 1 else None

    def step(raw, slots):
        a, y = torch.zeros(b, w.w_o.k, dtype=BF, device=dev), torch.zeros(b, w.w_o.k, device=dev)
        S.ssd_decode(raw[:, c.mw.left.columns:], w.x_at, w.dt_at, w.conv_w, w.conv_b, carried, w.dt_bias, w.a_log, w.skip,
                     spec.groups, slots, state, y, w.norm, 1e-5, spec.norm_groups, a)
        return [(a, w.w_o, c.mw.right_scale)]

    decode_against(c, step, lambda h: 1.3 * O.state_space(r, spec.to_json(), 1e-5, h), b, 8e-3)
    assert int((c.cache.state.abs().sum(1) > 0).sum()) == b


# ------------------------------------------------------------------ the model
def odd_cfg():
    """Widths and ranks that are not multiples of eight, single heads and groups, layers without feed-forward, top equal
    to the experts, one tap, one expert; latent widths of the decode kernel; rows read by two layers."""
    L, G, C, Z, T, X = LatentAttentionSpec, GlaSpec, ChunkedAttentionSpec, StateSpaceSpec, TwinNormLayerSpec, ChosenFfSpec
    lat = L(2, 64, 64, 72, 128, 0.1, 1e4, q_rank=30)
    return NugosunConfig(83, 100, [
        T(lat, X(3, 3, 50)), T(G(1, 72, 36, 1.0, 12), None), T(replace(lat, heads=3, dim=20, vdim=14, q_rank=9, kv_from=0), X(1, 1, 33)),
        T(PairSpec(C(5, 5, 12, 20, 0.3, RotarySpec(50.0, 2), 0.0, 1), Z(3, 10, 9, 3, 1, 5), -0.5, 2.0), SwigluFfSpec(70)),
        T(replace(lat, kv_from=0), None), T(G(5, 9, 13, 30.0, 20), SwigluFfSpec(33)),
        T(PairSpec(C(3, 1, 100, 36, 0.12, RotarySpec(1e6, 100, YARN), 2.0, 65), Z(1, 40, 64, 1, 9, 1), 1.0, 1.0), X(9, 2, 40))],
        1e-3, 0.7).validate()


def wide_cfg():
    """Head sizes outside the tensor-core attention kernels, attention without a chunk, big states."""
    C, Z, T = ChunkedAttentionSpec, StateSpaceSpec, TwinNormLayerSpec
    return NugosunConfig(65, 44, [
        T(PairSpec(C(2, 1, 136, 20, 0.1, RotarySpec(1e3, 64), 6.0, 0), Z(2, 150, 130, 2, 3, 2), 0.8, 0.9), SwigluFfSpec(30)),
        T(LatentAttentionSpec(2, 140, 16, 30, 40, 0.1, 1e3, q_rank=50), ChosenFfSpec(4, 2, 24)),
        T(GlaSpec(1, 144, 520, 3.0, 4), None)], 1e-4, 2.0).validate()


CFGS = {"tiny": M.nugosun_tiny, "odd": odd_cfg, "wide": wide_cfg}
TOL = {F32: 3e-5, BF: 0.2}


class Bench:
    """A random model with its plain counterpart; prompts' logits are computed once."""

    def __init__(self, dev, name, dtype):
        self.cfg = CFGS[name]()
        # bf16: the bias decides who is chosen, so that rounding cannot flip a close choice (the 32-bit runs and the
        # routing tests above leave it to the logits)
        self.tensors = {k: (v.float() * 30).to(BF) if dtype == BF and k.endswith("router.b") else v
                        for k, v in M.random_tensors(self.cfg, 11).items()}
        self.model = M.NugosunModel(M.build_weights(self.cfg, self.tensors, dev, dtype))
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
        eng = TwinNormDecode(bench.model, cache, max_batch=16, use_graph=use_graph)
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
