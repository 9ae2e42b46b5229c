"""Nugosun without a GPU: the plain restatement's mechanisms against hand-written loops (and planted mistakes that it
must show), configuration and checkpoint handling, the family registry, weight merging and padding, shared cache rows
and recurrent state, and the memory plan."""
import json
import math
from dataclasses import replace

import pytest
import torch
from oracle import nugosun as O

from rmlx_b200.cli.plan import plan, plan_nugosun, render
from rmlx_b200.config import (ChosenFfSpec, ChunkedAttentionSpec, ConfigError, GlaSpec, LatentAttentionSpec, NugosunConfig,
                              PairSpec, RodapelConfig, RotarySpec, SchedulerConfig, StateSpaceSpec, SwigluFfSpec,
                              TwinNormLayerSpec)
from rmlx_b200.models import nugosun as M
from rmlx_b200.models import registry
from rmlx_b200.ops import twin_norm as TN
from rmlx_b200.serve.engine import ServingEngine

D = torch.float64


def gen(seed):
    g = torch.Generator().manual_seed(seed)
    return lambda *s: torch.randn(*s, generator=g, dtype=D)


def rms(x, eps):
    return math.sqrt(sum(v * v for v in x) / len(x) + eps)


def silu(z):
    return z / (1 + math.exp(-z))


# ------------------------------------------------------------------ the oracle's mechanisms, by hand
def test_oracle_gated_linear_attention_by_hand():
    """The state written out as a sum over the past."""
    r = gen(1)
    heads, dim, vdim, rank, width, t, eps, tau = 2, 3, 5, 2, 6, 7, 1e-3, 3.0
    w = {"q": r(heads * dim, width), "k": r(heads * dim, width), "v": r(heads * vdim, width), "g": r(heads * vdim, width),
         "a1": r(rank, width), "a2": r(heads * dim, rank), "a2.b": r(heads * dim), "norm": r(vdim), "o": r(width, heads * vdim)}
    m = {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}
    h = r(t, width)
    got = O.gated_linear_attention(w, m, eps, h)
    alpha = torch.sigmoid((h @ w["a1"].T) @ w["a2"].T + w["a2.b"]) ** (1 / tau)
    for i in range(t):
        out = []
        for hd in range(heads):
            ks, vs = slice(hd * dim, (hd + 1) * dim), slice(hd * vdim, (hd + 1) * vdim)
            q, o = w["q"][ks] @ h[i] / math.sqrt(dim), torch.zeros(vdim, dtype=D)
            for j in range(i + 1):
                fade = torch.ones(dim, dtype=D)
                for s in range(j + 1, i + 1):
                    fade = fade * alpha[s, ks]
                o += float((q * fade * (w["k"][ks] @ h[j])).sum()) * (w["v"][vs] @ h[j])
            o = o / rms(o.tolist(), eps) * w["norm"]
            out += [float(a) * silu(float(b)) for a, b in zip(o, w["g"][vs] @ h[i])]
        assert torch.allclose(got[i], w["o"] @ torch.tensor(out, dtype=D), atol=1e-9)


def test_oracle_state_space_by_hand():
    r = gen(2)
    heads, vd, n, groups, taps, ng, width, t, eps = 4, 3, 2, 2, 3, 2, 6, 6, 1e-3
    inner, ch = heads * vd, heads * vd + 2 * groups * n
    w = {"in": r(inner + ch + heads, width), "conv": r(ch, taps), "conv.b": r(ch), "dt_bias": r(heads), "A_log": 0.3 * r(heads),
         "D": r(heads), "norm": r(inner), "o": r(width, inner)}
    m = {"heads": heads, "vdim": vd, "state": n, "groups": groups, "conv": taps, "norm_groups": ng}
    h = r(t, width)
    got = O.state_space(w, m, eps, h)
    raw = (h @ w["in"].T).tolist()
    state = [[[0.0] * vd for _ in range(n)] for _ in range(heads)]
    for i in range(t):
        c = []
        for k in range(ch):                                # the last tap is the current token's
            a = float(w["conv.b"][k])
            for j in range(taps):
                if i - j >= 0:
                    a += float(w["conv"][k, taps - 1 - j]) * raw[i - j][inner + k]
            c.append(silu(a))
        y = []
        for hd in range(heads):
            dt = math.log1p(math.exp(raw[i][inner + ch + hd] + float(w["dt_bias"][hd])))
            fade, g = math.exp(-math.exp(float(w["A_log"][hd])) * dt), hd // (heads // groups)
            for v in range(vd):
                x, o = c[hd * vd + v], 0.0
                for s in range(n):
                    state[hd][s][v] = fade * state[hd][s][v] + dt * c[inner + g * n + s] * x
                    o += state[hd][s][v] * c[inner + groups * n + g * n + s]
                y.append((o + float(w["D"][hd]) * x) * silu(raw[i][hd * vd + v]))
        size, out = inner // ng, []
        for g in range(ng):                                # the gate comes before the norm
            part = y[g * size:(g + 1) * size]
            out += [a / rms(part, eps) for a in part]
        assert torch.allclose(got[i], w["o"] @ (torch.tensor(out, dtype=D) * w["norm"]), atol=1e-9)


def test_oracle_chunked_attention_by_hand():
    r = gen(3)
    heads, groups, dim, vdim, width, t, eps, size = 4, 2, 6, 5, 6, 9, 1e-3, 4
    rot = {"base": 40.0, "dims": 4, "scaling": {"factor": 3.0, "original": 30.0, "fast": 4.0, "slow": 0.5}}
    m = {"heads": heads, "kv_heads": groups, "dim": dim, "vdim": vdim, "scale": 0.7, "softcap": 1.5, "mask": {"size": size}, "rot": rot}
    w = {}
    for n, rows in (("q", heads * dim), ("k", groups * dim), ("v", groups * vdim)):
        w[n], w[n + ".b"] = r(rows, width), r(rows)
    w["o"] = r(width, heads * vdim)
    h = r(t, width)
    got = O.chunked_attention(w, m, eps, h)
    at = lambda turns: 4 * math.log(30.0 / (2 * math.pi * turns)) / (2 * math.log(40.0))    # noqa: E731
    lo, hi = max(math.floor(at(4.0)), 0), min(math.ceil(at(0.5)), 3)
    freq = []
    for i in range(2):
        f, ramp = 40.0 ** (-2 * i / 4), min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        freq.append(f / 3.0 * ramp + f * (1 - ramp))
    grow = 0.1 * math.log(3.0) + 1

    def turned(name, row, head, pos):
        x = (w[name][head * dim:(head + 1) * dim] @ row + w[name + ".b"][head * dim:(head + 1) * dim]).tolist()
        for i in range(2):
            c, s, u, v = math.cos(pos * freq[i]) * grow, math.sin(pos * freq[i]) * grow, x[i], x[i + 2]
            x[i], x[i + 2] = u * c - v * s, v * c + u * s
        n = rms(x, eps)
        return torch.tensor([v / n for v in x], dtype=D)

    for i in range(t):
        outs = []
        for hd in range(heads):
            g = hd // (heads // groups)
            q, num, den = turned("q", h[i], hd, i), torch.zeros(vdim, dtype=D), 0.0
            for j in range(i // size * size, i + 1):
                z = float(q @ turned("k", h[j], g, j)) * 0.7
                e = math.exp(1.5 * math.tanh(z / 1.5))
                num += e * (w["v"][g * vdim:(g + 1) * vdim] @ h[j] + w["v.b"][g * vdim:(g + 1) * vdim])
                den += e
            outs.append(num / den)
        assert torch.allclose(got[i], w["o"] @ torch.cat(outs), atol=1e-9)


def test_oracle_latent_queries_and_routing_by_hand():
    r = gen(4)
    heads, dim, rot, vdim, rank, qr, width, t, eps = 2, 4, 4, 3, 5, 3, 6, 5, 1e-3
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "q_rank": qr, "scale": 0.4,
         "rot": {"base": 50.0, "dims": rot}}
    w = {"dq": r(qr, width), "dq.norm": r(qr), "uq": r(heads * (dim + rot), qr), "dkv": r(rank + rot, width), "dkv.norm": r(rank),
         "uk": r(heads * dim, rank), "uv": r(heads * vdim, rank), "o": r(width, heads * vdim)}
    h = r(t, width)
    got = O.latent_attention(w, m, eps, h, O.latent_rows(w, m, eps, h))

    def turn(x, pos):
        x = x.tolist()
        for p in range(2):
            a = pos * 50.0 ** (-2 * p / 4)
            u, v = x[2 * p], x[2 * p + 1]
            x[2 * p], x[2 * p + 1] = u * math.cos(a) - v * math.sin(a), v * math.cos(a) + u * math.sin(a)
        return torch.tensor(x, dtype=D)

    for i in range(t):
        outs = []
        for hd in range(heads):
            cq = w["dq"] @ h[i]
            q = w["uq"][hd * 8:(hd + 1) * 8] @ (cq / rms(cq.tolist(), eps) * w["dq.norm"])
            num, den = torch.zeros(vdim, dtype=D), 0.0
            for j in range(i + 1):
                down = w["dkv"] @ h[j]
                c = down[:rank] / rms(down[:rank].tolist(), eps) * w["dkv.norm"]
                e = math.exp(0.4 * float(q[:4] @ (w["uk"][hd * 4:(hd + 1) * 4] @ c) + turn(q[4:], i) @ turn(down[rank:], j)))
                num, den = num + e * (w["uv"][hd * vdim:(hd + 1) * vdim] @ c), den + e
            outs.append(num / den)
        assert torch.allclose(got[i], w["o"] @ torch.cat(outs), atol=1e-9)
    router, bias = r(6, width), 2 * r(6)
    idx, wt = O.route(router, bias, 2, h)
    for i in range(t):
        z = [float(router[e] @ h[i] + bias[e]) for e in range(6)]
        best = sorted(range(6), key=lambda e: -z[e])[:2]
        assert idx[i].tolist() == best
        assert abs(float(wt[i, 0]) - math.exp(z[best[0]]) / (math.exp(z[best[0]]) + math.exp(z[best[1]]))) < 1e-12


def test_rotary_frequencies_match_the_restatement():
    for rot in ({"base": 300000.0, "dims": 28}, {"base": 1e4, "dims": 2},
                {"base": 70000.0, "dims": 36, "scaling": {"factor": 6.0, "original": 1500.0, "fast": 20.0, "slow": 1.5}},
                {"base": 50.0, "dims": 64, "scaling": {"factor": 8.0, "original": 4.0, "fast": 1.0, "slow": 0.9}},
                {"base": 1e4, "dims": 40, "scaling": {"factor": 1.0, "original": 2048.0, "fast": 32.0, "slow": 1.0}}):
        f, grow = TN.rotary_frequencies(rot["base"], rot["dims"], rot.get("scaling"))
        want, g = O.turn_frequencies(rot)
        assert torch.allclose(f, torch.tensor(want, dtype=D), rtol=1e-12) and abs(grow - g) < 1e-12


def test_oracle_prefix_does_not_depend_on_what_follows():
    cfg = M.nugosun_tiny()
    w = {k: v.double() for k, v in M.random_tensors(cfg, 3).items()}
    toks = torch.randint(0, cfg.vocab_size, (60,), generator=torch.Generator().manual_seed(2)).tolist()
    full = O.forward(cfg.to_json(), w, toks)
    assert torch.allclose(full[:41], O.forward(cfg.to_json(), w, toks[:41]), atol=1e-10)


PARTS = ["chunk", "softcap", "rotation", "yarn", "bias", "decay", "tau", "conv", "step", "skip", "norm groups", "left", "right",
         "router bias", "query norm", "shared rows", "embedding", "norm offset", "key groups"]


@pytest.mark.parametrize("part", PARTS)
def test_a_planted_mistake_shows_in_the_logits(part):
    """The random weights of the other tests do not hide a fault in any single mechanism."""
    cfg = M.nugosun_tiny()
    w = {k: v.double() for k, v in M.random_tensors(cfg, 11).items()}
    toks = torch.randint(0, cfg.vocab_size, (60,), generator=torch.Generator().manual_seed(5)).tolist()
    c = cfg.to_json()
    want = O.forward(c, w, toks)
    bad, wb = json.loads(json.dumps(c)), dict(w)
    mix = [layer["mixer"] for layer in bad["layers"]]
    if part == "chunk":
        mix[2]["left"]["mask"]["size"] += 1
    elif part == "softcap":
        mix[2]["left"]["softcap"] = 1.0
    elif part == "rotation":
        mix[1]["rot"]["base"] *= 2
        mix[3]["rot"]["base"] *= 2
    elif part == "yarn":
        mix[2]["left"]["rot"].pop("scaling")
    elif part == "bias":
        wb["l2.mix.left.k.b"] = w["l2.mix.left.k.b"] * 0
    elif part == "decay":
        wb["l0.mix.a2.b"] = w["l0.mix.a2.b"] - 2
    elif part == "tau":
        mix[0]["tau"] = 1.0
    elif part == "conv":
        wb["l2.mix.right.conv"] = torch.roll(w["l2.mix.right.conv"], 1, 1)
    elif part == "step":
        wb["l2.mix.right.dt_bias"] = w["l2.mix.right.dt_bias"] + 1
    elif part == "skip":
        wb["l2.mix.right.D"] = w["l2.mix.right.D"] * 0
    elif part == "norm groups":
        mix[2]["right"]["norm_groups"] = 1
    elif part in ("left", "right"):
        mix[2][part + "_scale"] = 1.0
    elif part == "router bias":
        wb["l0.mlp.router.b"] = w["l0.mlp.router.b"] * 0
    elif part == "query norm":
        wb["l1.mix.dq.norm"] = torch.ones_like(w["l1.mix.dq.norm"])
    elif part == "shared rows":
        mix[3].pop("kv_from")
        wb.update({k.replace("l1.mix.dkv", "l3.mix.dkv"): v.roll(1, 0) for k, v in w.items() if "l1.mix.dkv" in k})
    elif part == "embedding":
        bad["embedding"]["scale"] = 1.0
    elif part == "norm offset":
        wb["l1.norm2"] = w["l1.norm2"] - 1
    else:
        wb["l2.mix.right.in"] = w["l2.mix.right.in"].clone()
        lo = 2 * 96                                        # B of the two groups change places
        wb["l2.mix.right.in"][lo:lo + 40] = w["l2.mix.right.in"][lo:lo + 40].roll(20, 0)
    err = (O.forward(bad, wb, toks) - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    assert float(err.max()) > 1e-2


# ------------------------------------------------------------------ configuration, checkpoints, registry
def test_config_round_trip_and_errors():
    cfg = M.nugosun_tiny()
    c = cfg.to_json()
    back = NugosunConfig.from_json(json.loads(json.dumps(c)))
    back.layers[0].mixer.decay_rank = cfg.layers[0].mixer.decay_rank        # comes with the weights
    assert back == cfg and back.num_layers == 5 and back.hidden_size == cfg.width
    for path, value in ((("layers", 0, "type"), "conv"), (("layers", 2, "mixer", "left", "kv_heads"), 4),
                        (("layers", 2, "mixer", "left", "rot", "dims"), 7), (("layers", 2, "mixer", "left", "rot", "dims"), 34),
                        (("layers", 0, "mlp", "router", "top"), 8), (("layers", 1, "mlp", "kind"), "glu"), (("norm", "eps"), 0.0),
                        (("layers", 0, "mlp", "router", "experts"), 300),
                        (("layers", 0, "mixer", "dim"), 300), (("layers", 0, "mixer", "tau"), 0.0),
                        (("layers", 2, "mixer", "right", "groups"), 4), (("layers", 2, "mixer", "right", "norm_groups"), 5),
                        (("layers", 2, "mixer", "right", "state"), 0), (("layers", 2, "mixer", "right", "conv"), 0),
                        (("layers", 3, "mixer", "kv_from"), 0), (("layers", 3, "mixer", "kv_from"), 3),
                        (("layers", 3, "mixer", "kv_rank"), 70), (("layers", 3, "mixer", "rot", "base"), 1.0),
                        (("layers", 1, "mixer", "q_rank"), 0), (("layers", 2, "mixer", "left", "rot", "scaling", "factor"), 0.0)):
        bad = json.loads(json.dumps(c))
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ConfigError):
            NugosunConfig.from_json(bad)
    chain = json.loads(json.dumps(c))                       # rows that are themselves another layer's
    chain["layers"].append(json.loads(json.dumps(chain["layers"][3])))
    chain["layers"][5]["mixer"]["kv_from"] = 3
    with pytest.raises(ConfigError):
        NugosunConfig.from_json(chain)
    plain = json.loads(json.dumps(c))
    plain["layers"][4]["mixer"]["left"].update(mask=None, softcap=None)     # neither chunks nor a cap
    left = NugosunConfig.from_json(plain).layers[4].mixer.left
    assert left.chunk == 0 and left.softcap == 0.0 and left.rot.scaling is None
    from rmlx_b200.models.rodapel import rodapel_tiny
    other = rodapel_tiny().to_json()                        # a family without query latents refuses them
    other["layers"][2]["mixer"]["q_rank"] = 16
    with pytest.raises(ConfigError):
        RodapelConfig.from_json(other)


def test_registry_picks_the_family_and_loads_a_checkpoint(tmp_path):
    cfg = M.nugosun_tiny()
    tensors = M.random_tensors(cfg, 1)
    M.save_checkpoint(str(tmp_path), cfg, tensors)
    fam = registry.family_of(registry.read_json(str(tmp_path)))
    assert fam.name == "nugosun" and fam.kernels == "twin_norm"
    model = registry.from_pretrained(str(tmp_path), device="cpu", dtype=torch.float32)
    assert isinstance(model, M.NugosunModel) and model.cfg.layers[0].mixer.decay_rank == 6
    assert torch.equal(model.w.embed, tensors["embed"].float()) and model.w.lm_head.w is model.w.embed
    with pytest.raises(KeyError):
        M.build_weights(cfg, {k: v for k, v in tensors.items() if k != "l0.mlp.e3.up"})
    with pytest.raises(ValueError):
        M.build_weights(cfg, {**tensors, "l1.mix.uk": tensors["l1.mix.uk"][1:]})
    with pytest.raises(ValueError):
        M.build_weights(cfg, tensors, dtype=torch.float16)
    from rmlx_b200._lib import NativeError
    with pytest.raises(NativeError):                        # no CPU path
        model.forward(torch.tensor([1, 2]))


def test_kernel_set_holds_every_launcher_the_family_calls():
    """A checkout in which nothing is built compiles the family's sources alone: what its operations call must be there."""
    import re

    from rmlx_b200 import _build
    sources = "".join((_build.CSRC / s).read_text() for s in _build.SETS["twin_norm"]["cuda"])
    have = set(re.findall(r'extern "C" [a-z ]+(rmlx_\w+)\(', sources))
    need = set()
    for name in ("scan", "twin_norm", "routed", "post_norm", "parallel_block", "latent", "gemm"):
        need |= set(re.findall(r"\.(rmlx_\w+)\(", (_build.ROOT / "ops" / f"{name}.py").read_text()))
    assert need - have == set()


def test_weights_are_merged_padded_and_spread():
    T = TwinNormLayerSpec
    lat = LatentAttentionSpec(3, 10, 6, 11, 21, 0.2, 100.0, q_rank=13)
    pair = PairSpec(ChunkedAttentionSpec(4, 2, 12, 5, 0.3, RotarySpec(100.0, 4), 2.0, 7), StateSpaceSpec(3, 5, 6, 1, 3, 1), 0.5, 2.0)
    cfg = NugosunConfig(50, 20, [T(lat, SwigluFfSpec(9)), T(GlaSpec(3, 7, 5, 2.0, 5), ChosenFfSpec(3, 2, 10)), T(pair, None),
                                 T(replace(lat, heads=2, kv_from=0), None)], 1e-4).validate()
    t = {k: v.float() for k, v in M.random_tensors(cfg, 2).items()}
    w = M.build_weights(cfg, t, dtype=torch.float32)
    h = torch.zeros(2, 24)
    h[:, :20] = torch.randn(2, 20)
    x = h[:, :20]
    eq = lambda a, b: torch.testing.assert_close(a, b, atol=1e-5, rtol=1e-5)                # noqa: E731
    eq(w.layers[0].norm1[:20], 1 + t["l0.norm1"])
    assert not w.layers[0].norm1[20:].any() and not w.final_norm[20:].any() and w.embed.shape == (50, 24)
    a = w.layers[0].mix
    raw = h @ a.w_in.w.T
    eq(raw[:, :13], x @ t["l0.mix.dq"].T)
    assert a.down_at == 16 and not raw[:, 13:16].any() and a.source == 0
    eq(raw[:, 16:43], x @ t["l0.mix.dkv"].T)
    c = torch.zeros(2, 16)
    c[:, :13] = torch.randn(2, 13)
    eq((c @ a.w_uq.w.T)[:, :48], c[:, :13] @ t["l0.mix.uq"].T)
    shared = w.layers[3].mix
    assert shared.source == 0 and shared.c_norm is None and shared.w_in.n == 16
    g = w.layers[1].mix
    raw = h @ g.w_in.w.T
    at = g.at
    for name, lo, n in (("q", at[0], 21), ("k", at[1], 21), ("v", at[2], 15), ("g", at[3], 15), ("a1", at[4], 5)):
        assert lo % 8 == 0
        eq(raw[:, lo:lo + n], x @ t[f"l1.mix.{name}"].T)
    eq((raw[:, at[4]:at[4] + 16] @ g.w_a2.T)[:, :21], (x @ t["l1.mix.a1"].T) @ t["l1.mix.a2"].T)
    eq(g.norm, t["l1.mix.norm"].repeat(3))
    f = w.layers[1].mlp
    assert f.w_gu.w.shape == (3, 128, 24) and f.w_down.w.shape == (3, 128, 64) and f.spec.limit == 0.0
    eq(f.correction, t["l1.mlp.router.b"])
    p = w.layers[2].mix
    raw = h @ p.w_in.w.T
    eq(raw[:, :48], x @ t["l2.mix.left.q"].T)
    eq(raw[:, 72:82], x @ t["l2.mix.left.v"].T)
    eq(p.left.bias, torch.cat([t[f"l2.mix.left.{n}.b"] for n in "qkv"]))
    right, inp = raw[:, p.left.columns:], x @ t["l2.mix.right.in"].T
    eq(right[:, :15], inp[:, :15])
    eq(right[:, p.right.x_at:p.right.x_at + 27], inp[:, 15:42])
    eq(right[:, p.right.dt_at:p.right.dt_at + 3], inp[:, 42:])
    eq(p.right.conv_w, t["l2.mix.right.conv"].T)
    assert float(p.left_scale.unique()) == 0.5 and float(p.right_scale.unique()) == 2.0
    o = torch.randn(2, 4, 5)
    spread = torch.zeros(2, 4, 8)
    spread[..., :5] = o
    eq((spread.reshape(2, -1) @ p.left.w_o.w.T)[:, :20], o.reshape(2, -1) @ t["l2.mix.left.o"].T)
    assert w.nbytes() > sum(v.numel() * 4 for k, v in t.items() if v.dim() == 2 and "conv" not in k)


# ------------------------------------------------------------------ cache, engine, plan
def test_cache_holds_rows_and_states_per_layer():
    cfg = M.nugosun_tiny()
    model = M.NugosunModel(M.build_weights(cfg, M.random_tensors(cfg, 1), dtype=torch.float32))
    c = model.new_cache(9, max_seqs=3)
    assert [k is None for k in c.k] == [True, False, False, True, False]    # layer 3 reads layer 1's rows
    assert c.v[1] is c.k[1] and c.k[1].shape == (9, 1, 16, 72 + 16 + 8)
    assert c.k[2].shape[3] == 32 and c.v[2].shape[3] == 48
    assert c.layer_state(0, "gla").shape == (4, 3, 24, 40) and c.layer_state(2, "ssd").shape == (4, 6, 20, 16)
    conv = c.layer_state(2, "conv")
    assert conv.shape == (4, 3, 96 + 2 * 2 * 20) and conv.stride(0) == c.state.stride(0)
    a = c.add_sequence(0)
    conv[a], c.layer_state(4, "conv")[a] = 2.0, 3.0
    b = c.fork(0, 1)
    assert torch.equal(c.state[a], c.state[b]) and float(conv[b].min()) == 2.0
    c.free_sequence(0)
    assert c.add_sequence(2) == a and not c.state[a].any()  # a slot that is used again starts at zero
    with pytest.raises(ValueError):
        c.trim(1, 1)
    one_tap = NugosunConfig(11, 16, [TwinNormLayerSpec(PairSpec(
        ChunkedAttentionSpec(1, 1, 8, 8, 1.0, RotarySpec(10.0, 8)), StateSpaceSpec(1, 4, 4, 1, 1, 1)))], 1e-5).validate()
    assert list(M.state_shapes(one_tap)[0]) == ["ssd"]


def test_engine_refuses_a_prefix_cache_over_recurrent_layers():
    cfg = M.nugosun_tiny()
    model = M.NugosunModel(M.build_weights(cfg, M.random_tensors(cfg, 1), dtype=torch.float32))
    with pytest.raises(ValueError, match="recurrent"):
        ServingEngine(model, 20, SchedulerConfig(max_batch_size=2), use_prefix_cache=True)
    with pytest.raises(ValueError):
        model.new_cache(4, kv_quant="q8")
    with pytest.raises(ValueError):
        model.make_decode_engine(model.new_cache(4), 1, comm=object())
    eng = ServingEngine(model, 20, SchedulerConfig(max_batch_size=2))
    assert eng.cache.state.shape[0] == 3 and eng.cache.max_blocks_per_seq == 19
    eng.close_sequence(eng.open_sequence())


def test_memory_plan():
    p = plan("nugosun-4096", weights="bf16", batch=4, ctx=8192)
    states = M.state_shapes(M.nugosun_4096())
    gla, ssd = 16 * 128 * 256, 64 * 128 * 64 + 3 * (4096 + 2 * 128)
    assert p["state_bytes_per_sequence"] == 4 * (8 * gla + 8 * ssd) and len([s for s in states if s]) == 16 and p["fits"]
    assert p["kv_bytes_per_token_per_gpu"] == 8 * (512 + 64 + 8) * 2 + 8 * 8 * 256 * 2   # shared rows are held once
    assert p["kv_bytes_needed"] == 4 * (8192 * p["kv_bytes_per_token_per_gpu"] + p["state_bytes_per_sequence"])
    assert p["weight_bytes_per_gpu"]["lm_head"] == 0 and "recurrent state" in render(p)
    with pytest.raises(ValueError):
        plan("nugosun-4096", weights="q4")
    small = plan_nugosun(cfg=M.nugosun_tiny())
    assert small["fits"] and small["model"] == "nugosun"
