"""Nizorax without a GPU: the plain restatement's mechanisms against hand-written loops (and planted mistakes that it must
show), configuration and checkpoint handling, the family registry, weight merging and padding, cache rows and state per
layer run, and the memory plan."""
import json
import math

import pytest
import torch
from oracle import nizorax as O

from rmlx_b200.cli.plan import plan, plan_nizorax, render
from rmlx_b200.config import (ConfigError, DifferentialAttentionSpec, GroupedFfSpec, LightningSpec, LoopSpec, NizoraxConfig,
                              PolyNormFfSpec, RotarySpec, SandwichLayerSpec, SchedulerConfig)
from rmlx_b200.models import nizorax as M
from rmlx_b200.models import registry
from rmlx_b200.ops import twin_norm as TN
from rmlx_b200.serve.engine import ServingEngine

D = torch.float64


def gen(seed):
    g = torch.Generator().manual_seed(seed)
    return lambda *s: torch.randn(*s, generator=g, dtype=D)


def rms(x, eps):
    return math.sqrt(sum(v * v for v in x) / len(x) + eps)


def sigmoid(z):
    return 1 / (1 + math.exp(-z))


# ------------------------------------------------------------------ the oracle's mechanisms, by hand
def test_oracle_differential_attention_by_hand():
    r = gen(3)
    heads, groups, dim, vdim, width, t, eps, window, diff = 4, 2, 6, 5, 6, 9, 1e-3, 4, 0.3
    rot = {"base": 40.0, "dims": 4, "scaling": {"factor": 3.0, "original": 30.0, "high": 4.0, "low": 0.5}}
    m = {"heads": heads, "kv_heads": groups, "dim": dim, "vdim": vdim, "scale": 0.7, "diff": diff, "mask": {"size": window}, "rot": rot}
    w = {"q": r(heads * 2 * dim, width), "k": r(groups * 2 * dim, width), "v": r(groups * vdim, width), "o": r(width, heads * vdim)}
    w.update({n: 0.3 * r(dim) for n in ("lq1", "lk1", "lq2", "lk2")})
    h = r(t, width)
    got = O.differential_attention(w, m, eps, h)
    freq = []
    for i in range(2):
        f = 40.0 ** (-2 * i / 4)
        wave = 2 * math.pi / f
        if wave < 30.0 / 4.0:
            freq.append(f)
        elif wave > 30.0 / 0.5:
            freq.append(f / 3.0)
        else:
            s = (30.0 / wave - 0.5) / (4.0 - 0.5)
            freq.append((1 - s) * f / 3.0 + s * f)
    lam = math.exp(float(w["lq1"] @ w["lk1"])) - math.exp(float(w["lq2"] @ w["lk2"])) + diff

    def turned(name, row, part, pos):
        x = (w[name][part * dim:(part + 1) * dim] @ row).tolist()
        for i in range(2):
            c, s, u, v = math.cos(pos * freq[i]), math.sin(pos * freq[i]), x[2 * i], x[2 * i + 1]
            x[2 * i], x[2 * i + 1] = u * c - v * s, v * c + u * s
        return torch.tensor(x, dtype=D)

    for i in range(t):
        outs = []
        for hd in range(heads):
            g, maps = hd // (heads // groups), []
            for a in (0, 1):                               # a head's rows are its first map's, then its second's
                num, den = torch.zeros(vdim, dtype=D), 0.0
                for j in range(max(0, i - window + 1), i + 1):
                    e = math.exp(0.7 * float(turned("q", h[i], hd * 2 + a, i) @ turned("k", h[j], g * 2 + a, j)))
                    num, den = num + e * (w["v"][g * vdim:(g + 1) * vdim] @ h[j]), den + e
                maps.append(num / den)
            o = maps[0] - lam * maps[1]
            outs.append(o / rms(o.tolist(), eps) * (1 - diff))
        assert torch.allclose(got[i], w["o"] @ torch.cat(outs), atol=1e-9)


def test_oracle_lightning_attention_by_hand():
    """The state written out as a sum over the past."""
    r = gen(1)
    heads, dim, vdim, width, t, eps = 2, 3, 5, 6, 7, 1e-3
    w = {"q": r(heads * dim, width), "k": r(heads * dim, width), "v": r(heads * vdim, width), "g": r(heads * vdim, width),
         "norm": r(heads * vdim), "o": r(width, heads * vdim)}
    m, h = {"heads": heads, "dim": dim, "vdim": vdim, "decay": [0.6, 0.95]}, r(t, width)
    got = O.lightning(w, m, eps, h)
    act = lambda name, i: [float(z) * sigmoid(float(z)) for z in w[name] @ h[i]]              # noqa: E731
    for i in range(t):
        out = []
        for hd in range(heads):
            q, o = act("q", i)[hd * dim:(hd + 1) * dim], [0.0] * vdim
            for j in range(i + 1):
                k, v = act("k", j)[hd * dim:(hd + 1) * dim], act("v", j)[hd * vdim:(hd + 1) * vdim]
                s = m["decay"][hd] ** (i - j) * sum(a * b for a, b in zip(q, k))
                o = [a + s * b for a, b in zip(o, v)]
            out += o
        n, gate = rms(out, eps), [sigmoid(float(z)) for z in w["g"] @ h[i]]      # all heads are normed together
        y = [a / n * float(b) * c for a, b, c in zip(out, w["norm"], gate)]
        assert torch.allclose(got[i], w["o"] @ torch.tensor(y, dtype=D), atol=1e-9)


def test_oracle_norm_convolution_and_activation_by_hand():
    r = gen(2)
    x, w, b, eps = 3 * r(4, 7) + 5, r(7), r(7), 1e-2
    got = O.layer_norm(x, eps, w, b)
    for i in range(4):
        row = x[i].tolist()
        mean = sum(row) / 7
        dev = math.sqrt(sum((v - mean) ** 2 for v in row) / 7 + eps)
        assert torch.allclose(got[i], torch.tensor([(v - mean) / dev for v in row], dtype=D) * w + b, atol=1e-12)
    for taps in (1, 2, 4):
        c = r(7, taps)
        got = O.short_conv(x, c)
        for i in range(4):
            for k in range(7):
                y = float(x[i, k])
                for j in range(taps):                      # the last tap is the current token's
                    at = i - taps + 1 + j
                    y += float(c[k, j]) * float(x[at, k]) if at >= 0 else 0.0
                assert abs(float(got[i, k]) - y) < 1e-12
    act = r(4)
    got = O.poly_norm(x, eps, act)
    for i in range(4):
        row = x[i].tolist()
        n = [rms([v ** p for v in row], eps) for p in (1, 2, 3)]
        want = [sum(float(act[p]) * v ** (p + 1) / n[p] for p in range(3)) + float(act[3]) for v in row]
        assert torch.allclose(got[i], torch.tensor(want, dtype=D), atol=1e-10)


def test_oracle_routing_and_shared_expert_by_hand():
    r = gen(4)
    e, top, count, keep, width, ff = 12, 3, 4, 2, 6, 5
    spec, router, h = {"experts": e, "top": top, "scale": 1.4, "groups": {"count": count, "keep": keep}}, r(e, width), r(20, width)
    idx, wt = O.route(router, spec, h)
    differs = 0
    for i in range(20):
        s = [sigmoid(float(router[j] @ h[i])) for j in range(e)]
        best = [sum(sorted(s[g * 3:(g + 1) * 3])[-2:]) for g in range(count)]
        kept = sorted(range(count), key=lambda g: -best[g])[:keep]
        pick = sorted((j for j in range(e) if j // 3 in kept), key=lambda j: -s[j])[:top]
        assert idx[i].tolist() == pick and torch.allclose(wt[i], torch.tensor([1.4 * s[j] for j in pick], dtype=D), atol=1e-12)
        differs += sorted(pick) != sorted(sorted(range(e), key=lambda j: -s[j])[:top])
    assert differs > 3                                     # the groups matter
    w = {"router": router, "shared.gate": r(7, width), "shared.up": r(7, width), "shared.down": r(width, 7)}
    for j in range(e):
        w.update({f"e{j}.gate": r(ff, width), f"e{j}.up": r(ff, width), f"e{j}.down": r(width, ff)})
    got = O.expert_mix(w, {"router": spec, "expert": {"ff": ff}, "shared": {"ff": 7}}, h)

    def glu(p, x):
        return w[p + "down"] @ torch.tensor([float(a) * sigmoid(float(a)) * float(b) for a, b in zip(w[p + "gate"] @ x, w[p + "up"] @ x)], dtype=D)

    for i in range(20):
        y = glu("shared.", h[i])
        for j, a in zip(idx[i].tolist(), wt[i]):
            y = y + a * glu(f"e{j}.", h[i])
        assert torch.allclose(got[i], y, atol=1e-9)


def test_layer_order_with_a_loop():
    layers = [None] * 5
    assert O.runs({"layers": layers}) == [0, 1, 2, 3, 4]
    assert O.runs({"layers": layers, "loop": {"start": 1, "stop": 3, "times": 3}}) == [0, 1, 2, 1, 2, 1, 2, 3, 4]
    assert O.runs({"layers": layers, "loop": {"start": 4, "stop": 5, "times": 1}}) == [0, 1, 2, 3, 4]
    for loop in (None, LoopSpec(1, 3, 3), LoopSpec(0, 5, 2), LoopSpec(4, 5, 1)):
        cfg = M.nizorax_tiny()
        cfg.layers, cfg.loop = cfg.layers + cfg.layers[:1], loop
        assert cfg.validate().runs == O.runs(cfg.to_json()) and cfg.num_layers == len(cfg.runs)


def test_rotary_frequencies_match_the_restatement():
    for rot in ({"base": 300000.0, "dims": 28}, {"base": 1e4, "dims": 2}, {"base": 1e4, "dims": 0},
                {"base": 70000.0, "dims": 36, "scaling": {"factor": 6.0, "original": 1500.0, "high": 20.0, "low": 1.5}},
                {"base": 50.0, "dims": 64, "scaling": {"factor": 8.0, "original": 4.0, "high": 1.0, "low": 0.9}},
                {"base": 1e4, "dims": 40, "scaling": {"factor": 1.0, "original": 2048.0, "high": 32.0, "low": 1.0}}):
        f, grow = TN.rotary_frequencies(rot["base"], rot["dims"], rot.get("scaling"))
        assert torch.allclose(f, torch.tensor(O.turn_frequencies(rot), dtype=D), rtol=1e-12) and grow == 1.0


def test_oracle_prefix_does_not_depend_on_what_follows():
    cfg = M.nizorax_tiny()
    w = {k: v.double() for k, v in M.random_tensors(cfg, 3).items()}
    toks = torch.randint(0, cfg.vocab_size, (60,), generator=torch.Generator().manual_seed(2)).tolist()
    full = O.forward(cfg.to_json(), w, toks)
    assert torch.allclose(full[:41], O.forward(cfg.to_json(), w, toks[:41]), atol=1e-10)


PARTS = ["window", "rotation", "scaling", "neighbours", "difference", "diff", "map order", "decay", "gate", "mixer norm",
         "convolution", "second convolution", "loop", "activation", "router scale", "groups", "shared", "norm bias", "output norm",
         "output bias", "embedding", "logits", "key groups"]


@pytest.mark.parametrize("part", PARTS)
def test_a_planted_mistake_shows_in_the_logits(part):
    """The random weights of the other tests do not hide a fault in any single mechanism."""
    cfg = M.nizorax_tiny()
    w = {k: v.double() for k, v in M.random_tensors(cfg, 11).items()}
    toks = torch.randint(0, cfg.vocab_size, (60,), generator=torch.Generator().manual_seed(5)).tolist()
    c = cfg.to_json()
    want = O.forward(c, w, toks)
    bad, wb = json.loads(json.dumps(c)), dict(w)
    mix = [layer["mixer"] for layer in bad["layers"]]
    if part == "window":
        mix[1]["mask"]["size"] += 1
    elif part == "rotation":
        mix[1]["rot"]["base"] *= 2
    elif part == "scaling":
        mix[1]["rot"].pop("scaling")
    elif part == "neighbours":                             # pairs of halves instead: the same rows in another order
        half = torch.cat([torch.arange(0, 40, 2), torch.arange(1, 40, 2)])
        for n, parts in (("q", 6), ("k", 6)):
            wb[f"l3.mix.{n}"] = w[f"l3.mix.{n}"].view(parts, 40, -1)[:, half].reshape(parts * 40, -1)
    elif part == "difference":
        wb["l1.mix.lq1"] = w["l1.mix.lq1"] + 1.0
    elif part == "diff":
        mix[3]["diff"] += 0.2
    elif part == "map order":
        wb["l1.mix.q"] = w["l1.mix.q"].view(6, 2, 28, -1).flip(1).reshape(w["l1.mix.q"].shape)
        wb["l1.mix.k"] = w["l1.mix.k"].view(2, 2, 28, -1).flip(1).reshape(w["l1.mix.k"].shape)
    elif part == "decay":
        mix[0]["decay"][2] = 0.95
    elif part == "gate":
        wb["l2.mix.g"] = w["l2.mix.g"] * 0
    elif part == "mixer norm":
        wb["l0.mix.norm"] = torch.ones_like(w["l0.mix.norm"])
    elif part in ("convolution", "second convolution"):
        n = "l1.canon1" if part == "convolution" else "l1.canon2"
        wb[n] = torch.roll(w[n], 1, 1)
    elif part == "loop":
        bad["loop"]["times"] = 3
    elif part == "activation":
        wb["l1.mlp.act"] = w["l1.mlp.act"] * torch.tensor([1.0, 1.0, 1.0, 0.0], dtype=D)
    elif part == "router scale":
        bad["layers"][0]["mlp"]["router"]["scale"] = 1.0
    elif part == "groups":
        bad["layers"][0]["mlp"]["router"]["groups"]["keep"] = 3
    elif part == "shared":
        wb["l0.mlp.shared.down"] = w["l0.mlp.shared.down"] * 0
    elif part == "norm bias":
        wb["l2.norm1.b"] = w["l2.norm1.b"] * 0
    elif part == "output norm":
        wb["l2.norm1b"] = torch.ones_like(w["l2.norm1b"])
    elif part == "output bias":
        wb["l3.norm2b.b"] = w["l3.norm2b.b"] * 0
    elif part == "embedding":
        bad["embedding"]["scale"] = 1.0
    elif part == "logits":
        bad["logit_scale"] = 1.0
    else:                                                  # the groups' keys change places
        wb["l1.mix.k"] = w["l1.mix.k"].roll(56, 0)
    err = (O.forward(bad, wb, toks) - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    assert float(err.max()) > 1e-2


# ------------------------------------------------------------------ configuration, checkpoints, registry
def test_config_round_trip_and_errors():
    cfg = M.nizorax_tiny()
    c = cfg.to_json()
    assert NizoraxConfig.from_json(json.loads(json.dumps(c))) == cfg and cfg.num_layers == 6 and cfg.hidden_size == cfg.width
    for path, value in ((("layers", 0, "type"), "conv"), (("layers", 1, "mixer", "kv_heads"), 4),
                        (("layers", 1, "mixer", "rot", "dims"), 7), (("layers", 1, "mixer", "rot", "dims"), 30),
                        (("layers", 0, "mlp", "router", "top"), 5), (("layers", 1, "mlp", "kind"), "glu"), (("norm", "eps"), 0.0),
                        (("layers", 0, "mlp", "router", "experts"), 300), (("layers", 0, "mlp", "router", "groups", "count"), 4),
                        (("layers", 0, "mlp", "router", "groups", "keep"), 0), (("layers", 0, "mlp", "router", "groups", "keep"), 4),
                        (("layers", 0, "mixer", "dim"), 300), (("layers", 0, "mixer", "decay"), [0.5]),
                        (("layers", 1, "mixer", "rot", "scaling", "factor"), 0.0), (("layers", 1, "mixer", "rot", "scaling", "low"), 3.0),
                        (("loop", "start"), 3), (("loop", "stop"), 5), (("loop", "times"), 0), (("canon", "taps"), 0)):
        bad = json.loads(json.dumps(c))
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ConfigError):
            NizoraxConfig.from_json(bad)
    plain = json.loads(json.dumps(c))
    plain["layers"][1]["mixer"].update(mask=None, rot=None)                 # neither a window nor a rotation
    plain["layers"][0]["mlp"]["router"].update(groups=None)
    plain.update(loop=None)
    back = NizoraxConfig.from_json(plain)
    assert back.layers[1].mixer.window == 0 and back.layers[1].mixer.rot.dims == 0 and back.loop is None and back.runs == [0, 1, 2, 3]
    assert back.layers[0].mlp.groups == 1 and NizoraxConfig.from_json(back.to_json()) == back


def test_shared_experts_are_cut_into_slices_as_wide_as_the_routed_ones():
    for f, want in ((GroupedFfSpec(6, 2, 40, shared=56), (2, 40)), (GroupedFfSpec(6, 2, 40, shared=40), (1, 40)),
                    (GroupedFfSpec(6, 2, 40), (0, 40)), (GroupedFfSpec(6, 2, 40, shared=7), (1, 40)),
                    (GroupedFfSpec(40, 31, 8, shared=100), (1, 100)), (GroupedFfSpec(40, 28, 8, shared=100), (4, 25))):
        assert f.validate().slices == want and want[0] * want[1] >= f.shared


def test_registry_picks_the_family_and_loads_a_checkpoint(tmp_path):
    cfg = M.nizorax_tiny()
    tensors = M.random_tensors(cfg, 1)
    M.save_checkpoint(str(tmp_path), cfg, tensors)
    fam = registry.family_of(registry.read_json(str(tmp_path)))
    assert fam.name == "nizorax" and fam.kernels == "sandwich"
    model = registry.from_pretrained(str(tmp_path), device="cpu", dtype=torch.float32)
    assert isinstance(model, M.NizoraxModel) and model.cfg == cfg
    assert torch.equal(model.w.embed, tensors["embed"].float()) and torch.equal(model.w.lm_head.w, tensors["head"].float())
    with pytest.raises(KeyError):
        M.build_weights(cfg, {k: v for k, v in tensors.items() if k != "l0.mlp.shared.up"})
    with pytest.raises(ValueError):
        M.build_weights(cfg, {**tensors, "l1.canon2": tensors["l1.canon2"][:, 1:]})
    with pytest.raises(ValueError):
        M.build_weights(cfg, tensors, dtype=torch.float16)
    from rmlx_b200._lib import NativeError
    with pytest.raises(NativeError):                        # no CPU path
        model.forward(torch.tensor([1, 2]))


def test_kernel_set_holds_every_launcher_the_family_calls():
    """A checkout in which nothing is built compiles the family's sources alone: what its operations call must be there."""
    import re

    from rmlx_b200 import _build
    sources = "".join((_build.CSRC / s).read_text() for s in _build.SETS["sandwich"]["cuda"])
    have = set(re.findall(r'extern "C" [a-z ]+(rmlx_\w+)\(', sources))
    need = set()
    for name in ("sandwich", "routed", "parallel_block", "gemm"):
        need |= set(re.findall(r"\.(rmlx_\w+)\(", (_build.ROOT / "ops" / f"{name}.py").read_text()))
    need |= {"rmlx_rotary_norm_append", "rmlx_lightning_scan", "rmlx_scan_record", "rmlx_gated_norm", "rmlx_lightning_step",
             "rmlx_postnorm_in", "rmlx_matvec_out", "rmlx_postnorm_max_rows", "rmlx_gated_act", "rmlx_sgemm"}
    assert need - have == set()


def test_weights_are_merged_padded_and_spread():
    T = SandwichLayerSpec
    attn = DifferentialAttentionSpec(4, 2, 10, 5, 0.3, RotarySpec(100.0, 4), 0.3, 7)
    cfg = NizoraxConfig(50, 20, [T(attn, PolyNormFfSpec(9)), T(LightningSpec(3, 7, 5, [0.5, 0.7, 0.9]), GroupedFfSpec(4, 2, 10, 2, 1, 2.0, 15)),
                                 T(attn, None)], 1e-4, logit_scale=0.3, taps=3, loop=LoopSpec(0, 2, 2)).validate()
    t = {k: v.float() for k, v in M.random_tensors(cfg, 2).items()}
    w = M.build_weights(cfg, t, dtype=torch.float32)
    h = torch.zeros(2, 24)
    h[:, :20] = torch.randn(2, 20)
    x = h[:, :20]
    eq = lambda a, b: torch.testing.assert_close(a, b, atol=1e-5, rtol=1e-5)                # noqa: E731
    assert len(w.layers) == 5 and w.layers[0] is w.layers[2] and w.layers[1] is w.layers[3]
    l0, l1 = w.layers[0], w.layers[1]
    eq(l0.norm1[:, :20], torch.stack([t["l0.norm1"], t["l0.norm1.b"]]))
    eq(l0.post2[:, :20], torch.stack([t["l0.norm2b"], t["l0.norm2b.b"]]))
    assert not l0.norm1[:, 20:].any() and w.layers[4].norm2 is None and w.layers[4].conv2 is None
    eq(l0.conv1[:, :20], t["l0.canon1"].t())
    eq(l1.conv2[:, :20], t["l1.canon2"].t())
    eq(w.final_norm[:, :20], 0.3 * torch.stack([t["final.norm"], t["final.norm.b"]]))       # carries the logits' factor
    raw = h @ l0.mix.w_in.w.T
    eq(raw[:, :80], x @ t["l0.mix.q"].T)
    eq(raw[:, 80:120], x @ t["l0.mix.k"].T)
    eq(raw[:, 120:130], x @ t["l0.mix.v"].T)
    lam = torch.exp(t["l0.mix.lq1"] @ t["l0.mix.lk1"]) - torch.exp(t["l0.mix.lq2"] @ t["l0.mix.lk2"]) + 0.3
    assert abs(l0.mix.diff.weight - float(lam)) < 1e-5 and abs(l0.mix.diff.scale - 0.7) < 1e-12 and l0.mix.diff.eps == 1e-4
    o = torch.randn(2, 4, 5)
    spread = torch.zeros(2, 4, 8)
    spread[..., :5] = o
    eq((spread.reshape(2, -1) @ l0.mix.w_o.w.T)[:, :20], o.reshape(2, -1) @ t["l0.mix.o"].T)
    raw, at = h @ l1.mix.w_in.w.T, l1.mix.at
    for name, lo, n in (("q", at[0], 21), ("k", at[1], 21), ("v", at[2], 15), ("g", at[3], 15)):
        assert lo % 8 == 0
        eq(raw[:, lo:lo + n], x @ t[f"l1.mix.{name}"].T)
    eq((h @ l0.mlp.w_up.w.T)[:, :9], x @ t["l0.mlp.up"].T)
    assert l0.mlp.w_up.w.shape == (64, 24) and not l0.mlp.w_down.w[:, 9:].any()
    f = l1.mlp                                              # four routed experts, then the shared one in two slices
    assert f.always == 2 and f.w_gu.w.shape == (6, 128, 24) and f.w_down.w.shape == (6, 128, 64) and f.correction is None
    parts = sum((torch.nn.functional.silu(h @ f.w_gu.w[e, :64].T) * (h @ f.w_gu.w[e, 64:].T)) @ f.w_down.w[e].T for e in (4, 5))
    eq(parts[:, :20], (torch.nn.functional.silu(x @ t["l1.mlp.shared.gate"].T) * (x @ t["l1.mlp.shared.up"].T)) @ t["l1.mlp.shared.down"].T)
    once = M.build_weights(NizoraxConfig(50, 20, cfg.layers, 1e-4, taps=3).validate(), t, dtype=torch.float32)
    assert w.nbytes() == once.nbytes() > sum(v.numel() * 4 for k, v in t.items() if v.dim() == 2 and "canon" not in k)


# ------------------------------------------------------------------ cache, engine, plan
def test_cache_holds_rows_and_states_per_run():
    cfg = M.nizorax_tiny()
    model = M.NizoraxModel(M.build_weights(cfg, M.random_tensors(cfg, 1), dtype=torch.float32))
    c = model.new_cache(9, max_seqs=3)
    assert [k is None for k in c.k] == [True, False, True, False, True, False]           # layers 1 and 2 run twice
    assert c.k[1].shape == (9, 2, 16, 64) and c.v[1].shape == (9, 2, 16, 56) and c.k[3].data_ptr() != c.k[1].data_ptr()
    assert c.k[5].shape == (9, 3, 16, 80) and c.v[5].shape == (9, 3, 16, 24)
    assert c.layer_state(0, "state").shape == (4, 3, 24, 40) and c.layer_state(4, "state").shape == (4, 2, 36, 16)
    assert c.layer_state(2, "state").data_ptr() != c.layer_state(4, "state").data_ptr()
    conv = c.layer_state(3, "conv2")
    assert conv.shape == (4, 2, 104) and conv.stride(0) == c.state.stride(0)
    with pytest.raises(KeyError):
        c.layer_state(2, "conv2")                           # a layer without feed-forward
    a = c.add_sequence(0)
    conv[a], c.layer_state(1, "conv2")[a] = 2.0, 3.0
    b = c.fork(0, 1)
    assert torch.equal(c.state[a], c.state[b]) and float(c.layer_state(3, "conv2")[b].min()) == 2.0
    c.free_sequence(0)
    assert c.add_sequence(2) == a and not c.state[a].any()  # a slot that is used again starts at zero
    with pytest.raises(ValueError):
        c.trim(1, 1)
    attn = DifferentialAttentionSpec(1, 1, 8, 8, 1.0, RotarySpec(10.0, 8), 0.5)
    one_tap = NizoraxConfig(11, 16, [SandwichLayerSpec(attn)], 1e-5, taps=1).validate()
    assert M.state_shapes(one_tap) == [None]


def test_engine_refuses_what_the_design_cannot_do():
    cfg = M.nizorax_tiny()
    model = M.NizoraxModel(M.build_weights(cfg, M.random_tensors(cfg, 1), dtype=torch.float32))
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
    p = plan("nizorax-4096", weights="bf16", batch=4, ctx=8192)
    assert p["state_bytes_per_sequence"] == 4 * (16 * 32 * 128 * 128 + 32 * 2 * 3 * 4096) and p["fits"]
    assert p["kv_bytes_per_token_per_gpu"] == 16 * 8 * (2 * 64 + 128) * 2
    assert p["kv_bytes_needed"] == 4 * (8192 * p["kv_bytes_per_token_per_gpu"] + p["state_bytes_per_sequence"])
    assert "recurrent state" in render(p)
    with pytest.raises(ValueError):
        plan("nizorax-4096", weights="q4")
    small = plan_nizorax(cfg=M.nizorax_tiny())
    assert small["fits"] and small["model"] == "nizorax"
    once = M.nizorax_tiny()
    once.loop = None
    a, b = small, plan_nizorax(cfg=once)                    # a loop holds no more weights but more cache, and reads more
    assert a["weight_bytes_per_gpu"] == b["weight_bytes_per_gpu"] and a["kv_bytes_per_token_per_gpu"] > b["kv_bytes_per_token_per_gpu"]
    assert a["decode_roofline"]["us_per_step"] > b["decode_roofline"]["us_per_step"]
