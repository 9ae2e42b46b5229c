"""Rodapel without a GPU: the plain restatement's mechanisms against hand-written loops (and planted mistakes
that it must show), configuration and checkpoint handling, the family registry, weight merging and padding,
the paged cache with recurrent state, ragged plans for latent and recurrent layers, and the memory plan."""
import json
import math

import pytest
import torch
from oracle import rodapel as O

from rmlx_b200.cli.plan import plan, render
from rmlx_b200.config import (ClampedFfSpec, ConfigError, LatentAttentionSpec, PostNormLayerSpec, RodapelConfig,
                              RoutedFfSpec, SchedulerConfig, WindowAttentionSpec, WkvSpec)
from rmlx_b200.kv.paged import PagedKvCache
from rmlx_b200.models import registry
from rmlx_b200.models import rodapel as M
from rmlx_b200.models.ragged import Entry, RaggedBatch
from rmlx_b200.serve.engine import ServingEngine

D = torch.float64


def gen(seed):
    g = torch.Generator().manual_seed(seed)
    return lambda *s: torch.randn(*s, generator=g, dtype=D)


def rms(x, eps):
    return math.sqrt(sum(v * v for v in x) / len(x) + eps)


# ------------------------------------------------------------------ the oracle's mechanisms, by hand
def test_oracle_window_attention_by_hand():
    r = gen(1)
    heads, groups, dim, vdim, width, t, window, eps = 4, 2, 3, 5, 6, 9, 4, 1e-3
    m = {"heads": heads, "kv_heads": groups, "dim": dim, "vdim": vdim, "scale": 0.7, "mask": {"size": window}}
    w = {"q": r(heads * dim, width), "k": r(groups * dim, width), "v": r(groups * vdim, width), "q.norm": r(dim),
         "k.norm": r(dim), "g": r(heads, width), "o": r(width, heads * vdim)}
    h = r(t, width)
    got = O.window_attention(w, m, eps, h)
    for i in range(t):
        outs = []
        for hd in range(heads):
            g = hd // (heads // groups)
            q = w["q"][hd * dim:(hd + 1) * dim] @ h[i]
            q = q / rms(q.tolist(), eps) * w["q.norm"]
            num, den = torch.zeros(vdim, dtype=D), 0.0
            for j in range(max(0, i - window + 1), i + 1):
                k = w["k"][g * dim:(g + 1) * dim] @ h[j]
                k = k / rms(k.tolist(), eps) * w["k.norm"]
                e = math.exp(float(q @ k) * 0.7)
                num += e * (w["v"][g * vdim:(g + 1) * vdim] @ h[j])
                den += e
            outs.append(num / den / (1 + math.exp(-float(w["g"][hd] @ h[i]))))
        assert torch.allclose(got[i], w["o"] @ torch.cat(outs), atol=1e-10)


def test_oracle_latent_attention_by_hand():
    r = gen(2)
    heads, dim, rot, vdim, rank, width, t, eps, base = 3, 4, 4, 5, 7, 6, 6, 1e-3, 50.0
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": 0.4,
         "rot": {"base": base, "dims": rot}}
    w = {"q": r(heads * (dim + rot), width), "dkv": r(rank + rot, width), "dkv.norm": r(rank), "uk": r(heads * dim, rank),
         "uv": r(heads * vdim, rank), "o": r(width, heads * vdim)}
    h = r(t, width)

    def turn(x, p):
        y = x.clone()
        for i in range(rot // 2):
            a = p * base ** (-2 * i / rot)
            y[2 * i] = x[2 * i] * math.cos(a) - x[2 * i + 1] * math.sin(a)
            y[2 * i + 1] = x[2 * i + 1] * math.cos(a) + x[2 * i] * math.sin(a)
        return y

    lat, key = [], []
    for j in range(t):
        d = w["dkv"] @ h[j]
        lat.append(d[:rank] / rms(d[:rank].tolist(), eps) * w["dkv.norm"])
        key.append(turn(d[rank:], j))
    got = O.latent_attention(w, m, eps, h)
    for i in range(t):
        outs = []
        for hd in range(heads):
            q = w["q"][hd * (dim + rot):(hd + 1) * (dim + rot)] @ h[i]
            num, den = torch.zeros(vdim, dtype=D), 0.0
            for j in range(i + 1):
                s = q[:dim] @ (w["uk"][hd * dim:(hd + 1) * dim] @ lat[j]) + turn(q[dim:], i) @ key[j]
                e = math.exp(float(s) * 0.4)
                num += e * (w["uv"][hd * vdim:(hd + 1) * vdim] @ lat[j])
                den += e
            outs.append(num / den)
        assert torch.allclose(got[i], w["o"] @ torch.cat(outs), atol=1e-10)


def test_oracle_recurrence_as_a_sum_over_the_past():
    """o_t = sum over s < t of (r_t . prod of decays . k_s) v_s, plus the bonus term."""
    r = gen(3)
    h, t, d = 2, 6, 3
    rr, k, v, u = r(h, t, d), r(h, t, d), r(h, t, d), r(h, d)
    w = torch.sigmoid(r(h, t, d))
    got = O.wkv_recurrence(rr, k, v, w, u)
    for hd in range(h):
        for i in range(t):
            want = float((rr[hd, i] * u[hd] * k[hd, i]).sum()) * v[hd, i]
            for s in range(i):
                decay = torch.ones(d, dtype=D)
                for q in range(s + 1, i):
                    decay = decay * w[hd, q]
                want = want + float((rr[hd, i] * decay * k[hd, s]).sum()) * v[hd, s]
            assert torch.allclose(got[hd, i], want, atol=1e-10)


def test_oracle_feed_forward_and_routing_by_hand():
    r = gen(4)
    gate, up, down, h = r(5, 4), r(5, 4), r(4, 5), 3 * r(6, 4)
    got = O.clamped_gate_ffn(gate, up, down, 1.5, h)
    for i in range(6):
        g, u = (gate @ h[i]).tolist(), (up @ h[i]).tolist()
        act = [min(a, 1.5) / (1 + math.exp(-1.702 * min(a, 1.5))) * (max(-1.5, min(b, 1.5)) + 1) for a, b in zip(g, u)]
        assert torch.allclose(got[i], down @ torch.tensor(act, dtype=D), atol=1e-12)
    mlp = {"router": {"experts": 3, "identity": 2, "top": 2}, "expert": {"limit": 1.5}}
    w = {"router": r(5, 4), "correction": r(5)}
    for e in range(3):
        w.update({f"e{e}.gate": r(5, 4), f"e{e}.up": r(5, 4), f"e{e}.down": r(4, 5)})
    got, some_identity, moved = O.expert_mix(w, mlp, h), False, False
    for i in range(6):
        s = torch.softmax(w["router"] @ h[i], 0)
        pick = sorted(range(5), key=lambda e: -float(s[e] + w["correction"][e]))[:2]
        some_identity |= any(e >= 3 for e in pick)
        moved |= set(pick) != set(sorted(range(5), key=lambda e: -float(s[e]))[:2])
        want = sum(s[e] * (h[i] if e >= 3 else O.clamped_gate_ffn(w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], 1.5,
                                                                  h[i:i + 1])[0]) for e in pick)
        assert torch.allclose(got[i], want, atol=1e-12)
    assert some_identity and moved


def test_oracle_prefix_does_not_depend_on_what_follows():
    cfg = M.rodapel_tiny()
    w = {k: v.double() for k, v in M.random_tensors(cfg, 3).items()}
    toks = torch.randint(0, cfg.vocab_size, (40,), generator=torch.Generator().manual_seed(2)).tolist()
    full = O.forward(cfg.to_json(), w, toks)
    assert torch.allclose(full[:31], O.forward(cfg.to_json(), w, toks[:31]), atol=1e-10)


@pytest.mark.parametrize("part", ["window", "decay", "bonus", "identity", "correction", "limit", "rotation", "gate"])
def test_a_planted_mistake_shows_in_the_logits(part):
    """The random weights of the other tests do not hide a fault in any single mechanism."""
    cfg = M.rodapel_tiny()
    w = {k: v.double() for k, v in M.random_tensors(cfg, 11).items()}
    toks = torch.randint(0, cfg.vocab_size, (60,), generator=torch.Generator().manual_seed(5)).tolist()
    c = cfg.to_json()
    want = O.forward(c, w, toks)
    bad, wb = json.loads(json.dumps(c)), dict(w)
    if part == "window":
        bad["layers"][1]["mixer"]["mask"]["size"] += 1
    elif part == "decay":
        wb["l0.mix.w0"] = w["l0.mix.w0"] + 0.5
    elif part == "bonus":
        wb["l0.mix.u"] = w["l0.mix.u"] * 0
    elif part == "identity":
        bad["layers"][1]["mlp"]["router"].update(experts=4, identity=4)     # two experts taken for identity
    elif part == "correction":
        wb["l1.mlp.correction"] = w["l1.mlp.correction"] * 0
    elif part == "limit":
        bad["layers"][0]["mlp"]["limit"] = 1.0
    elif part == "rotation":
        bad["layers"][2]["mixer"]["rot"]["base"] *= 2
    else:
        wb["l3.mix.g"] = w["l3.mix.g"] * 0
    err = (O.forward(bad, wb, toks) - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    assert float(err.max()) > 1e-2


# ------------------------------------------------------------------ configuration, checkpoints, registry
def test_config_round_trip_and_errors():
    cfg = M.rodapel_tiny()
    back = RodapelConfig.from_json(json.loads(json.dumps(cfg.to_json())))
    back.layers[0].mixer.decay_rank = cfg.layers[0].mixer.decay_rank        # comes with the weights
    assert back == cfg and back.num_layers == 4 and back.hidden_size == cfg.width
    c = cfg.to_json()
    for path, value in ((("layers", 0, "type"), "conv"), (("layers", 1, "mixer", "kv_heads"), 4),
                        (("layers", 2, "mixer", "rot", "dims"), 7), (("layers", 1, "mlp", "router", "top"), 9),
                        (("layers", 0, "mlp", "kind"), "glu"), (("norm", "eps"), 0.0), (("layers", 0, "mixer", "dim"), 300)):
        bad = json.loads(json.dumps(c))
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ConfigError):
            RodapelConfig.from_json(bad)
    plain = json.loads(json.dumps(c))
    plain["layers"][3]["mixer"]["mask"] = None                              # no window
    assert RodapelConfig.from_json(plain).layers[3].mixer.window == 0


def test_registry_picks_the_family_and_loads_a_checkpoint(tmp_path):
    cfg = M.rodapel_tiny()
    tensors = M.random_tensors(cfg, 1)
    M.save_checkpoint(str(tmp_path), cfg, tensors)
    assert registry.family_of(registry.read_json(str(tmp_path))).name == "rodapel"
    model = registry.from_pretrained(str(tmp_path), device="cpu", dtype=torch.float32)
    assert isinstance(model, M.RodapelModel) and model.cfg.layers[0].mixer.decay_rank == 8
    assert torch.equal(model.w.embed, tensors["embed"].float())
    with pytest.raises(KeyError):
        M.build_weights(cfg, {k: v for k, v in tensors.items() if k != "l1.mlp.e3.up"})
    with pytest.raises(ValueError):
        M.build_weights(cfg, {**tensors, "l2.mix.uk": tensors["l2.mix.uk"][1:]})
    with pytest.raises(ValueError):
        M.build_weights(cfg, tensors, dtype=torch.float16)
    from rmlx_b200._lib import NativeError
    with pytest.raises(NativeError):                                        # no CPU path
        model.forward(torch.tensor([1, 2]))


def test_weights_are_merged_padded_and_spread():
    A, L, K, P = WindowAttentionSpec, LatentAttentionSpec, WkvSpec, PostNormLayerSpec
    cfg = RodapelConfig(50, 20, [P(A(4, 2, 12, 5, 0.3, 7), ClampedFfSpec(9, 1.0)), P(L(3, 10, 6, 11, 21, 0.2, 100.0), None),
                                 P(K(3, 7, 5), RoutedFfSpec(3, 1, 2, 10, 2.0))], 1e-4).validate()
    t = {k: v.float() for k, v in M.random_tensors(cfg, 2).items()}
    w = M.build_weights(cfg, t, dtype=torch.float32)
    h = torch.zeros(2, 24)
    h[:, :20] = torch.randn(2, 20)
    x = h[:, :20]
    eq = lambda a, b: torch.testing.assert_close(a, b, atol=1e-5, rtol=1e-5)                # noqa: E731
    a = w.layers[0].mix
    raw = h @ a.w_in.w.T
    eq(raw[:, :48], x @ t["l0.mix.q"].T)
    eq(raw[:, a.gate_at:a.gate_at + 4], x @ t["l0.mix.g"].T)
    o = torch.randn(2, 4, 5)
    spread = torch.zeros(2, 4, 8)
    spread[..., :5] = o
    eq((spread.reshape(2, -1) @ a.w_o.w.T)[:, :20], o.reshape(2, -1) @ t["l0.mix.o"].T)
    f = w.layers[0].mlp
    gu = h @ f.w_gu.w.T
    eq(gu[:, :9], x @ t["l0.mlp.gate"].T)
    eq(gu[:, 64:73], x @ t["l0.mlp.up"].T)
    assert not gu[:, 9:64].any() and f.w_down.w.shape == (24, 64) and not f.w_down.w[20:].any()
    m = w.layers[1].mix
    c = torch.zeros(2, 24)
    c[:, :21] = torch.randn(2, 21)
    q = torch.randn(2, 3, 16)
    q[..., 10:] = 0
    eq(torch.einsum("bhd,hld->bhl", q, m.w_uk)[..., :21],
       torch.einsum("bhd,hdl->bhl", q[..., :10], t["l1.mix.uk"].view(3, 10, 21)))
    kv = (c @ m.w_ukv.w.T).view(2, 3, 16 + 16)
    eq(kv[..., :10], (c[:, :21] @ t["l1.mix.uk"].T).view(2, 3, 10))
    eq(kv[..., 16:27], (c[:, :21] @ t["l1.mix.uv"].T).view(2, 3, 11))
    assert not kv[..., 10:16].any() and torch.allclose(m.inv_freq, 100.0 ** (-torch.arange(3) / 3.0))
    k = w.layers[2].mix
    assert k.inner_p == 32 and k.rank_p == 16 and k.w_in.n == 4 * 32 + 16
    eq((h @ k.part(2).T)[:, :21], x @ t["l2.mix.v"].T)
    eq(torch.tanh(h @ k.part(4).T) @ k.w2.T[:, :21], torch.tanh(x @ t["l2.mix.w1"].T) @ t["l2.mix.w2"].T)
    e = w.layers[2].mlp
    assert e.w_gu.w.shape == (3, 128, 24) and e.w_down.w.shape == (3, 128, 64) and e.router.shape == (4, 24)
    eq((h @ e.w_gu.w[1].T)[:, 64:74], x @ t["l2.mlp.e1.up"].T)


# ------------------------------------------------------------------ cache, batches, engine
def test_paged_cache_with_recurrent_state():
    shapes = [(2, 8, 16), None, (1, 32, 0)]
    states = [None, {"wkv": (2, 3, 3), "prev": (8,)}, None]
    c = PagedKvCache(8, 3, 2, 8, dtype=torch.float32, max_seqs=3, max_blocks_per_seq=5, layer_shapes=shapes,
                     layer_states=states)
    assert c.k[1] is None and c.v[2] is c.k[2] and c.bytes_per_token() == (2 * 24 + 32) * 4
    wkv, prev = c.layer_state(1, "wkv"), c.layer_state(1, "prev")
    assert wkv.shape == (4, 2, 3, 3) and prev.shape == (4, 8) and prev.data_ptr() % 16 == 0 and c.idle_slot == 3
    assert c.bytes_per_sequence() == (20 + 8) * 4 and wkv.stride(0) == prev.stride(0) == c.state.stride(0)
    a = c.add_sequence(0)
    wkv[a], prev[a] = 1.5, -2.0
    c.reserve(0, 20)
    c.k[0][c.manager.block_table(0)[1]] = 3.0
    c.commit(0, 20)
    b = c.fork(0, 1)                                      # the child starts from the parent's state ...
    assert torch.equal(c.state[a], c.state[b])
    wkv[b] = 7.0                                          # ... and goes its own way
    assert float(wkv[a].max()) == 1.5
    c.reserve(1, 1)                                       # copy-on-write of a page, over layers without pages
    assert float(c.k[0][c.manager.block_table(1)[1]].max()) == 3.0
    with pytest.raises(ValueError):
        c.trim(0, 1)
    c.free_sequence(0)
    assert c.add_sequence(2) == a and not c.state[a].any()      # a slot that is used again starts at zero
    with pytest.raises(ValueError):
        c.adopt_prefix(2, [1], 16)
    with pytest.raises(ValueError):
        PagedKvCache(4, 3, 2, 8, layer_shapes=shapes, layer_states=states[:2])


def test_ragged_batch_plan_for_latent_and_recurrent_layers():
    ent = [Entry(7, [1] * 3, [2]), Entry(8, [2] * 40), Entry(9, [5], [0]), Entry(10, [6] * 5)]
    b = RaggedBatch(ent, [30, 10, 99, 0], [2, 0, 3, 1], heads=4, absorb=3).upload("cpu")
    assert b.runs.tolist() == [[0, 3, 2, 30], [3, 40, 0, 10], [43, 1, 3, 99], [44, 5, 1, 0]]
    assert b.absorbed.tolist() == [0, 1, 2, 43] and b.absorbed_len == 100
    # contexts of the entries with more than three tokens: 50 and 5 tokens
    assert b.ctx_pages.tolist() == [[0, 0], [0, 1], [0, 2], [0, 3], [1, 0]]
    rows = {tuple(t): c for t, c in zip(b.latent_tiles.tolist(), b.tile_ctx.tolist())}
    assert rows == {(3, 40, 10, 0): 0, (44, 5, 0, 1): 64}
    plain = RaggedBatch(ent, [30, 10, 99, 0], [2, 0, 3, 1], heads=4).upload("cpu")
    assert plain.latent_tiles is None and plain.absorbed is None and plain.single.tolist() == [43]


def test_engine_refuses_a_prefix_cache_over_recurrent_layers():
    cfg = M.rodapel_tiny()
    model = M.RodapelModel(M.build_weights(cfg, M.random_tensors(cfg, 1), dtype=torch.float32))
    with pytest.raises(ValueError, match="recurrent"):
        ServingEngine(model, 20, SchedulerConfig(max_batch_size=2), use_prefix_cache=True)
    with pytest.raises(ValueError):
        model.new_cache(4, kv_quant="q8")
    eng = ServingEngine(model, 20, SchedulerConfig(max_batch_size=2))
    assert eng.cache.state.shape[0] == 3 and eng.cache.max_blocks_per_seq == 19
    sid = eng.open_sequence()
    eng.close_sequence(sid)


def test_memory_plan():
    p = plan("rodapel-4096", weights="bf16", batch=4, ctx=8192)
    cfg = M.rodapel_4096()
    cache = M.state_shapes(cfg)
    assert p["state_bytes_per_sequence"] == sum(4 * (64 * 64 * 64 + 4096) for s in cache if s) and p["fits"]
    assert p["kv_bytes_needed"] == 4 * (8192 * p["kv_bytes_per_token_per_gpu"] + p["state_bytes_per_sequence"])
    assert "recurrent state" in render(p)
    with pytest.raises(ValueError):
        plan("rodapel-4096", weights="q4")
