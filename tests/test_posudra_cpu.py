"""Posudra without a GPU: the plain restatement's mechanisms against hand-written loops, configuration
and checkpoint handling, the family registry, weight padding, ragged-batch planning, the paged cache
with per-layer shapes, and the serving engine's mixed steps on a stub model."""
import json
import math

import pytest
import torch
from oracle import posudra as O

from rmlx_b200.config import (ConfigError, ParallelLayerSpec, PosudraConfig, SamplerConfig, SchedulerConfig,
                              ScoredAttentionSpec)
from rmlx_b200.kv.paged import OutOfBlocks, PagedKvCache
from rmlx_b200.models import posudra as M
from rmlx_b200.models import registry
from rmlx_b200.models.ragged import Entry, RaggedBatch, query_lanes, query_tiles
from rmlx_b200.models.weights import ParallelLayout
from rmlx_b200.serve.engine import ServingEngine


# ------------------------------------------------------------------ the oracle's mechanisms
def test_oracle_attention_by_hand():
    g = torch.Generator().manual_seed(1)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)     # noqa: E731
    heads, t, d, dv = 2, 5, 3, 4
    q, k, v = r(heads, t, d), r(heads, t, d), r(heads, t, dv)
    temp, r1, r2, sink = r(heads).abs() + 0.5, r(heads).abs(), r(heads).abs(), r(heads)
    got = O.scored_attention(q, k, v, 0.7, temp, 4.0, r1, r2, sink)
    for h in range(heads):
        for i in range(t):
            num, den = torch.zeros(dv, dtype=torch.float64), math.exp(sink[h])
            for j in range(i + 1):
                s = float(q[h, i] @ k[h, j]) * 0.7 * float(temp[h])
                s = 4.0 * math.tanh(s / 4.0) - float(r1[h]) * math.log(1 + float(r2[h]) * (i - j))
                num += math.exp(s) * v[h, j]
                den += math.exp(s)
            assert torch.allclose(got[h, i], num / den, atol=1e-12)


def test_oracle_activation_and_norm_by_hand():
    z = torch.tensor([-3.0, -0.5, 0.0, 0.5, 2.0], dtype=torch.float64)
    p, q = torch.tensor(0.3, dtype=torch.float64), torch.tensor(-0.8, dtype=torch.float64)
    ap, an = math.log1p(math.exp(0.3)), 0.5 + math.log1p(math.exp(-0.8))
    want = [ap * x * x + x / 2 if x > 0 else an * (math.exp(x) - 1 - x) + x / 2 for x in z.tolist()]
    assert torch.allclose(O.xielu(z, p, q), torch.tensor(want, dtype=torch.float64), atol=1e-12)
    x = torch.tensor([[3.0, 4.0]], dtype=torch.float64)
    assert torch.allclose(O.rms_norm(x, torch.tensor([1.0, 2.0]), 0.5), x / math.sqrt(13.0) * torch.tensor([1.0, 2.0]))


def test_oracle_prefix_does_not_depend_on_what_follows():
    cfg = M.posudra_tiny()
    w = M.random_tensors(cfg, 3)
    toks = torch.randint(0, cfg.vocab_size, (12,), generator=torch.Generator().manual_seed(2)).tolist()
    full = O.forward(cfg.to_json(), w, toks)
    assert torch.allclose(full[:7], O.forward(cfg.to_json(), w, toks[:7]), atol=1e-10)


# ------------------------------------------------------------------ configuration, checkpoints, registry
def test_config_round_trip_and_errors():
    cfg = M.posudra_tiny()
    assert PosudraConfig.from_json(json.loads(json.dumps(cfg.to_json()))) == PosudraConfig.from_json(cfg.to_json())
    j = cfg.to_json()
    j["layers"][0]["type"] = "recurrent"
    with pytest.raises(ConfigError):
        PosudraConfig.from_json(j)
    j = cfg.to_json()
    j["layers"][0]["mlp"]["kind"] = "experts"
    with pytest.raises(ConfigError):
        PosudraConfig.from_json(j)
    with pytest.raises(ConfigError):
        ScoredAttentionSpec(5, 2, 8, 8, 1.0).validate()
    assert cfg.num_layers == 3 and cfg.sliding_window == 0 and cfg.layers[1].ff == 0


def test_registry_picks_the_family_and_loads_a_checkpoint(tmp_path):
    cfg = M.posudra_tiny()
    tensors = M.random_tensors(cfg, 5)
    M.save_checkpoint(str(tmp_path), cfg, tensors)
    assert registry.family_of(registry.read_json(str(tmp_path))).name == "posudra"
    assert registry.family_of({"num_attention_heads": 4, "model_type": "qwen2"}).name == "transformer"
    with pytest.raises(ValueError):
        registry.family_of({"architecture": "unheard of"})
    for dt in (torch.float32, torch.bfloat16):
        model = registry.from_pretrained(str(tmp_path), "cpu", dt)
        assert isinstance(model, M.PosudraModel) and model.dtype == dt and model.cfg.num_layers == 3
    from rmlx_b200.loader.safetensors_loader import load_model
    weights, got = load_model(str(tmp_path))
    assert got.width == cfg.width and weights.layers[1].w_down is None
    with pytest.raises(Exception, match="CUDA"):
        cache = model.new_cache(4, max_seqs=1)
        cache.add_sequence(0)
        model.forward_batch([Entry(0, [1])], cache)          # no CPU path


def test_registry_transformer_family_unchanged(tmp_path):
    from rmlx_b200.config import tiny_dense_config
    from rmlx_b200.loader.safetensors_loader import save_checkpoint
    from rmlx_b200.models.transformer import TransformerModel
    from rmlx_b200.models.weights import random_state_dict
    cfg = tiny_dense_config()
    save_checkpoint(str(tmp_path), cfg, random_state_dict(cfg, 0))
    model = registry.from_pretrained(str(tmp_path), "cpu", torch.float32)
    assert type(model) is TransformerModel and model.cfg.num_layers == cfg.num_layers


def test_weights_are_merged_padded_and_spread():
    spec = ParallelLayerSpec(ScoredAttentionSpec(3, 1, 10, 5, 0.3, 8.0), 13)
    cfg = PosudraConfig(17, 21, [spec], 1e-5, 1.5).validate()
    t = M.random_tensors(cfg, 1, dtype=torch.float32)
    w = M.build_weights(cfg, t, "cpu", torch.float32).layers[0]
    assert w.n_raw == 64 and w.ff == 16 and tuple(w.w_in.w.shape) == (80, 24)      # 30 + 10 + 5 -> 64
    assert torch.equal(w.w_in.w[30:40, :21], t["l0.mix.k"]) and torch.equal(w.w_in.w[64:77, :21], t["l0.mlp.up"])
    assert not w.w_in.w[45:64].any() and not w.w_in.w[77:].any() and not w.w_in.w[:, 21:].any()
    assert tuple(w.w_o.w.shape) == (24, 24) and torch.equal(w.w_o.w[:21, 8:13], t["l0.mix.o"][:, 5:10])
    assert not w.w_o.w[:, 5:8].any() and not w.w_o.w[21:].any()
    assert w.norm1.dtype == torch.float32 and not w.norm1[21:].any() and not w.ls1[21:].any()
    assert w.act_p == pytest.approx(math.log1p(math.exp(float(t["l0.mlp.act"][0]))), rel=1e-6)
    assert w.act_n == pytest.approx(0.5 + math.log1p(math.exp(float(t["l0.mlp.act"][1]))), rel=1e-6)
    with pytest.raises(KeyError):
        M.build_weights(cfg, {k: v for k, v in t.items() if k != "l0.ls1"})
    with pytest.raises(ValueError):
        M.build_weights(cfg, {**t, "head": t["head"][:3]})
    with pytest.raises(ValueError):
        M.build_weights(cfg, t, dtype=torch.float16)


# ------------------------------------------------------------------ batches and caches
def test_ragged_batch_plan():
    b = RaggedBatch([Entry(7, [1, 2, 3], [2, 0]), Entry(9, [4]), Entry(8, list(range(300)), [299]), Entry(3, [5], [0])],
                    pos0=[10, 40, 0, 2], slots=[2, 0, 1, 3])
    assert b.num_tokens == 305 and b.starts == [0, 3, 4, 304] and b.single_host == [3, 304] and b.single_len == 41
    assert b.want_host == [2, 0, 303, 304]
    assert b.tiles_host == [(260, 44, 256, 1), (132, 128, 128, 1), (4, 128, 0, 1), (0, 3, 10, 2)]
    b.upload("cpu")
    assert b.tiles.tolist() == [list(t) for t in b.tiles_host] and b.tokens[3] == 4
    assert b.positions.tolist()[:4] == [10, 11, 12, 40] and b.token_seq.tolist()[2:5] == [2, 0, 1]
    assert b.single.tolist() == [3, 304] and b.want.tolist() == b.want_host
    for bad in ([], [Entry(0, [])], [Entry(0, [1]), Entry(0, [2])], [Entry(0, [1], [1])]):
        with pytest.raises(ValueError):
            RaggedBatch(bad, [0] * len(bad), list(range(len(bad))))


def test_query_tiles_cover_every_row_once():
    for lanes in (1, 2):
        lens = [1, 2, 127, 128, 129, 256, 257, 513]
        starts = [sum(lens[:i]) for i in range(len(lens))]
        rows = sorted(r for s, n, _, _ in query_tiles(starts, lens, [0] * 8, list(range(8)), 128 * lanes)
                      for r in range(s, s + n))
        assert rows == list(range(1, sum(lens)))          # the single token at row 0 is not a tile
    assert query_lanes([4096], 32) == 2 and query_lanes([4096], 4) == 1 and query_lanes([100] * 40, 32) == 1
    assert query_lanes([1] * 9, 64) == 1


def test_paged_cache_with_layer_shapes():
    shapes = [(2, 8, 16), (1, 24, 8)]
    c = PagedKvCache(6, 2, 2, 8, dtype=torch.float32, max_seqs=2, max_blocks_per_seq=5, layer_shapes=shapes)
    assert c.bytes_per_token() == (2 * 24 + 32) * 4
    c.add_sequence(0)
    c.add_sequence(1)
    data = {}
    for sid, n in ((0, 20), (1, 30)):
        c.reserve(sid, n)
        for l, (h, dk, dv) in enumerate(shapes):
            data[sid, l] = torch.randn(n, h, dk), torch.randn(n, h, dv)
            c.append(l, sid, *data[sid, l], 0)
        c.commit(sid, n)
    for (sid, l), (k, v) in data.items():
        assert torch.equal(c.get_keys(l, sid), k) and torch.equal(c.get_values(l, sid), v)
    with pytest.raises(OutOfBlocks):
        c.reserve(0, 40)
    c.free_sequence(1)
    c.reserve(0, 40)                                      # pages that were given back are used again
    with pytest.raises(ValueError):
        PagedKvCache(4, 2, 2, 64, kv_quant="q8", layer_shapes=shapes)
    with pytest.raises(ValueError):
        PagedKvCache(4, 3, 2, 8, layer_shapes=shapes)


# ------------------------------------------------------------------ serving engine, mixed steps
class StubModel:
    """A 'model' whose next token is (sum of everything its sequence has seen) mod vocab; it keeps the
    seen tokens itself and checks that the cache agrees about the position."""
    mixed_batches = True

    def __init__(self, vocab=50):
        self.cfg = M.posudra_tiny()
        self.vocab, self.device, self.layout = vocab, torch.device("cpu"), ParallelLayout()
        self.seen, self.batches = {}, []

    def new_cache(self, num_blocks, max_seqs=64, kv_quant=None, **_):
        return PagedKvCache(num_blocks, 1, 1, 8, max_seqs=max_seqs, max_blocks_per_seq=num_blocks - 1)

    def forward_batch(self, entries, cache):
        self.batches.append([(e.seq_id, len(e.tokens)) for e in entries])
        rows = []
        for e in entries:
            hist = self.seen.setdefault(e.seq_id, []) if cache.seq_len(e.seq_id) else \
                self.seen.__setitem__(e.seq_id, []) or self.seen[e.seq_id]
            assert len(hist) == cache.seq_len(e.seq_id)
            cache.reserve(e.seq_id, len(e.tokens))
            cache.commit(e.seq_id, len(e.tokens))
            for i, t in enumerate(e.tokens):
                hist.append(int(t))
                if i in set(e.want):
                    rows.append(torch.nn.functional.one_hot(torch.tensor(sum(hist) % self.vocab), self.vocab).float())
        return torch.stack(rows) if rows else torch.empty(0, self.vocab)

    def forward(self, toks, cache, ids, last_only=True):
        return self.forward_batch([Entry(s, [int(t)], [0]) for s, t in zip(ids, toks)], cache)


def _alone(prompt, n, vocab=50):
    hist, out = list(prompt), []
    for _ in range(n):
        out.append(sum(hist) % vocab)
        hist.append(out[-1])
    return out


@pytest.mark.parametrize("native", ["0", "1"])
def test_engine_mixes_prompt_chunks_with_decoded_tokens(native, monkeypatch):
    monkeypatch.setenv("RMLX_NATIVE_SERVING", native)
    model = StubModel()
    eng = ServingEngine(model, 40, SchedulerConfig(max_batch_size=3, max_prefill_chunk=8), SamplerConfig())
    prompts = [[3] * 5, [7] * 21, [1, 2], list(range(17)), [9]]
    ids = [eng.submit(p, 6) for p in prompts]
    out = eng.run_until_done()
    for sid, p in zip(ids, prompts):
        assert out[sid] == _alone(p, 6)
    # a prompt chunk and decoded tokens did share a batch
    assert any(len(b) > 1 and max(n for _, n in b) > 1 for b in model.batches)
    eng.step()                                            # evicts the last finished sequences
    assert eng.cache.manager.num_free_blocks() == 39


def test_engine_explicit_steps_and_trace_replay():
    from rmlx_b200.cli.trace import TraceReplay
    model = StubModel()
    eng = ServingEngine(model, 9, SchedulerConfig(max_batch_size=2))
    rep = TraceReplay(eng)
    free = eng.cache.manager.num_free_blocks()
    assert rep.step([{"id": "a", "tokens": [1, 2, 3], "want": []}]) is None
    got = rep.step([{"id": "b", "tokens": [5, 5], "want": [1]}, {"id": "a", "tokens": [4, 4], "want": [0, 1]}], ["b"])
    assert got.argmax(-1).tolist() == [10, 10, 14]        # b's sum, then a's running sums
    got = rep.step([{"id": "c", "tokens": [6], "want": [0]}, {"id": "a", "tokens": [1], "want": [0]}], ["a", "c"])
    assert got.argmax(-1).tolist() == [6, 15]
    assert eng.cache.manager.num_free_blocks() == free and not rep.seq_of
    sid = eng.open_sequence()
    with pytest.raises(ValueError):
        eng.run_entries([Entry(sid, [1]), Entry(sid, [2])])


def test_command_line_generate_on_the_transformer_family(tmp_path, capsys):
    from rmlx_b200.cli.main import main
    from rmlx_b200.config import tiny_dense_config
    from rmlx_b200.loader.safetensors_loader import save_checkpoint
    from rmlx_b200.models.weights import random_state_dict
    cfg = tiny_dense_config()
    save_checkpoint(str(tmp_path), cfg, random_state_dict(cfg, 0))
    assert main(["generate", "--model", str(tmp_path), "--device", "cpu", "--dtype", "float32", "--prompt", "1,2,3",
                 "--prompt", "4", "--steps", "3"]) == 0
    toks = json.loads(capsys.readouterr().out)["tokens"]
    model = registry.from_pretrained(str(tmp_path), "cpu", torch.float32)
    assert toks[0] == model.generate_greedy(torch.tensor([1, 2, 3]), 3) and len(toks[1]) == 3


def test_engine_explicit_steps_on_the_transformer_family():
    from rmlx_b200.config import tiny_dense_config
    from rmlx_b200.models.transformer import TransformerModel
    from rmlx_b200.models.weights import from_state_dict, random_state_dict
    cfg = tiny_dense_config()
    model = TransformerModel(from_state_dict(cfg, random_state_dict(cfg, 0), dtype=torch.float32))
    eng = ServingEngine(model, 20, SchedulerConfig(max_batch_size=2))
    a, b = eng.open_sequence(), eng.open_sequence()
    toks = list(range(7, 27))
    want = model.forward(torch.tensor(toks))
    got = [eng.run_entries([Entry(a, toks[:9], range(9)), Entry(b, [1, 2], ())])]
    got += [eng.run_entries([Entry(b, [3], ()), Entry(a, toks[9:], range(11))])]
    assert torch.allclose(torch.cat(got), want, atol=1e-4)


def test_kernel_sets_name_existing_sources_and_give_way_to_the_full_library(monkeypatch, tmp_path):
    from rmlx_b200 import _build, _lib
    for name, kinds in _build.SETS.items():
        for sources in kinds.values():
            assert all((_build.CSRC / s).exists() for s in sources), name
    built = []
    monkeypatch.setattr(_build, "LIB", tmp_path)
    monkeypatch.setattr(_build, "CUDA_LIB", tmp_path / "full.so")
    monkeypatch.setattr(_build, "build", lambda kinds, only="all": built.append((kinds, only)) or
                        {k: _build.set_lib(k, only) for k in kinds})
    monkeypatch.setattr(_lib, "_kernel_set", "all")
    _lib.prefer_kernels("parallel_block")
    assert _lib._library("cuda").name == "librmlx_b200_cuda_parallel_block.so"
    (tmp_path / "full.so").touch()
    assert _lib._library("cuda").name == "full.so" and built == [(("cuda",), "parallel_block")]
