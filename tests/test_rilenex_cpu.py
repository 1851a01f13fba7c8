"""Rilenex on the host: configuration, weight reader, block and slot bookkeeping, ragged batches, scheduling, and the plain
oracle against itself. The kernels are covered by ``test_gpu_rilenex.py``."""
import json
import random

import numpy as np
import pytest
import torch

import rilenex_oracle as oracle
from rilenex_common import CONFIGS, ODD, RANKS, attn, config, delta, hgrn2, make_model, make_weights, parallel
from sneppx_alg_b200.hub.formats import save_safetensors
from sneppx_alg_b200.hub.model_hub import ModelHub
from sneppx_alg_b200.models import ModelConfig, build_model, config_from_name, list_models
from sneppx_alg_b200.ops.gemm import XIELU, gemm
from sneppx_alg_b200.ops.ragged import RaggedBatch
from sneppx_alg_b200.serving.hybrid_runner import HybridRunner
from sneppx_alg_b200.serving.kv_cache import ChunkedKVCache
from sneppx_alg_b200.serving.llm_engine import LLMEngine, SamplingParams


# ------------------------------------------------------------------ configuration and weights
@pytest.mark.parametrize("name", list(CONFIGS))
def test_config_reads_and_round_trips(name, tmp_path):
    cfg = ModelConfig.from_dict(CONFIGS[name])
    c = CONFIGS[name]
    assert cfg.architecture == "rilenex" and cfg.vocab_size == c["vocab"] and cfg.hidden_size == c["width"]
    assert cfg.rms_norm_eps == c["norm"]["eps"] and cfg.num_hidden_layers == len(c["layers"]) == len(cfg.layer_specs)
    assert not cfg.validate()
    cfg.to_json(str(tmp_path / "c.json"))
    assert ModelConfig.from_json(str(tmp_path / "c.json")) == cfg


@pytest.mark.parametrize("fmt", ["safetensors", "sneppx"])
def test_weights_load_from_a_folder_and_save_back(tmp_path, fmt):
    W = make_weights(ODD)
    (tmp_path / "config.json").write_text(json.dumps(ODD))
    save_safetensors(str(tmp_path / "model.safetensors"), {k: v.bfloat16() for k, v in W.items()})
    model = ModelHub.from_pretrained(str(tmp_path), dtype=torch.float32)
    sd = model.to_reference_state_dict()
    assert set(sd) == set(W)
    for k in W:
        assert torch.equal(sd[k], W[k]), k
    assert model.config.estimate_parameters() == sum(t.numel() for t in sd.values())
    out = ModelHub.save_pretrained(model, str(tmp_path / "again"), fmt=fmt)
    again = ModelHub.from_pretrained(out, dtype=torch.float32).to_reference_state_dict()
    assert all(torch.equal(again[k].float(), sd[k]) for k in sd)


def test_ranks_come_from_the_tensors():
    model = make_model(ODD, make_weights(ODD))
    assert {(s["mixer"]["right"]["decay_rank"], s["mixer"]["right"]["gate_rank"])
            for s in model.config.layer_specs if s["type"] == "parallel"} == {RANKS}
    assert "decay_rank" not in ODD["layers"][1]["mixer"]["right"]      # the caller's configuration is left alone


def test_reader_refuses_missing_and_misshapen_tensors():
    W = make_weights(ODD)
    model = make_model(ODD, W)
    with pytest.raises(KeyError):
        model.load_reference_state_dict({k: v for k, v in W.items() if k != "l1.mix.left.talk"})
    with pytest.raises(ValueError):
        model.load_reference_state_dict({**W, "head": W["head"][:, :-1]})
    with pytest.raises(ValueError):
        build_model(ModelConfig.from_dict(config(16, 8, [{"type": "other", "mixer": {}, "mlp": None}])))


def test_reload_refreshes_the_activation():
    W = make_weights(ODD)
    model = make_model(ODD, W)
    before = model.layers[0].mlp.activation().a
    model.load_reference_state_dict({**W, "l0.mlp.act": torch.tensor([2.0, -1.0])})
    assert model.layers[0].mlp.activation().a != before


def test_presets():
    assert set(list_models()["rilenex"]) == {"tiny", "1B", "7B"}
    cfg = config_from_name("rilenex-tiny")
    assert build_model(cfg).config.estimate_parameters() == cfg.estimate_parameters()
    assert 1.2e9 < config_from_name("rilenex-1b").estimate_parameters() < 1.8e9


def test_kernels_are_required():
    model = make_model(ODD, make_weights(ODD))
    with pytest.raises(RuntimeError):
        model(torch.zeros(1, 3, dtype=torch.long))


# ------------------------------------------------------------------ activation
def test_xielu_matches_its_definition():
    z = torch.linspace(-8, 8, 401, dtype=torch.float64)
    for p, q in ((0.3, -0.7), (-3.0, 2.0), (0.0, 0.0)):
        want = oracle.xielu(z, torch.tensor(p, dtype=torch.float64), torch.tensor(q, dtype=torch.float64))
        assert torch.allclose(XIELU(p, q)(z), want, atol=1e-12)
    x, w = torch.randn(5, 8), torch.randn(6, 8)
    got = gemm(x, w, act=XIELU(0.3, -0.7))
    want = oracle.xielu((x @ w.T).double(), torch.tensor(0.3).double(), torch.tensor(-0.7).double())
    assert torch.allclose(got.double(), want, atol=1e-5)


# ------------------------------------------------------------------ block pool and slots
@pytest.mark.parametrize("sizes,bs", [((24,), 16), ((7, 40), 16), ((16, 64), 4), ((100,), 16), ((5,), 8), ((33, 47, 90), 10)])
def test_chunked_cache_keeps_exactly_the_visible_positions(sizes, bs):
    rng = random.Random(0)
    cache = ChunkedKVCache([(1, 2, 2)], sizes, 64, bs, dtype=torch.float32, device="cpu")
    store, owner = {}, {}
    for seq in range(3):
        cache.add_sequence(seq)
    for _ in range(120):
        seq = rng.randrange(3)
        n, p0 = rng.choice([1, 1, 1, 2, 3, 17, 90]), cache.lens[seq]
        for size in sizes:      # what the portion's first token still sees is there
            for p, e in zip(range(p0 // size * size, p0), cache.entries(seq, p0 // size * size, p0)):
                assert store[e] == (seq, p)
        entries = cache.reserve(seq, n)
        last = p0 + n - 1
        for p, e in zip(range(p0, p0 + n), entries):
            assert (e >= 0) == (p >= min(last // s * s for s in sizes))
            if e >= 0:
                store[e] = (seq, p)
        assert len(cache.tables[seq]) <= cache.table_width
        assert len(cache.tables[seq]) <= cache.blocks_for(10 ** 9)
        live = [b for t in cache.tables.values() for b in t]
        assert len(set(live)) == len(live) and len(live) + cache.pool.num_free == 64
    for seq in range(3):
        cache.free_sequence(seq)
    assert cache.pool.num_free == 64


def test_cache_without_attention_layers_uses_no_blocks():
    cache = ChunkedKVCache([], [], 1, 16, dtype=torch.float32, device="cpu")
    for seq in range(3):
        cache.add_sequence(seq)
        for n in (1, 15, 16, 40, 1):
            assert cache.reserve(seq, n) == [-1] * n
    assert cache.pool.num_free == 1 and cache.table_width == 0 and cache.blocks_for(100) == 0


def test_slots_are_handed_back():
    model = make_model(ODD, make_weights(ODD))
    cache = model.init_cache(2)
    assert [tuple(t.shape) for t in cache.k] and cache.k[0].shape[2:] == (2, 24) and cache.v[0].shape[2:] == (2, 20)
    cache.add_sequence(7)
    cache.add_sequence(8)
    with pytest.raises(MemoryError):
        cache.add_sequence(9)
    first = cache.slots[7]
    cache.free_sequence(7)
    cache.add_sequence(9)
    assert cache.slots[9] == first
    cache.free_sequence(7)      # not there any more: nothing happens
    with pytest.raises(NotImplementedError):
        cache.fork(8, 10)


# ------------------------------------------------------------------ ragged batches
def test_prompt_batch_layout():
    b = RaggedBatch.prompt("cpu", [[5, 6, 7], [8], [9] * 20], [0, 30, 2], [3, 0, 1], [[1, 2, 3], [4], list(range(10, 30))],
                           {24: [[], [50, 51, 52, 53, 54, 55], [60, 61]]}, [2, 3, 23], tile_rows=8)
    assert b.T == 24 and b.n == 3 and b.cu.tolist() == [0, 3, 4, 24] and b.pos0.tolist() == [0, 30, 2]
    assert b.tok_seq.tolist() == [0] * 3 + [1] + [2] * 20 and b.tok_pos.tolist() == [0, 1, 2, 30] + list(range(2, 22))
    v = b.views[24]
    assert v.rows == 24 + 6 + 2 and v.kv_row.tolist() == [0, 1, 2, 9] + list(range(12, 32))
    assert v.kv_base.tolist() == [0, 9 - 30, 12 - 2]
    assert v.gather_entry.tolist() == [50, 51, 52, 53, 54, 55, 60, 61] and v.gather_row.tolist() == [3, 4, 5, 6, 7, 8, 10, 11]
    assert v.tiles.view(-1, 2).tolist() == [[0, 0], [1, 0], [2, 0], [2, 8], [2, 16]]
    assert b.chunk_seq.tolist() == [0, 1, 2, 2] and b.chunk_start.tolist() == [0, 0, 0, 16] and b.chunk_first.tolist() == [0, 1, 2, 4]
    assert b.want.tolist() == [2, 3, 23]


def test_decode_batch_padding():
    lay, n = RaggedBatch.decode_layout(4, 3)
    host = torch.full((n,), 9, dtype=torch.int32)
    RaggedBatch.fill_decode(host.numpy(), 4, 3, [7, 8], [20, 31], [1, 0], [100, 200], [[5, 6], [7]], [1, 1])
    b = RaggedBatch.decode_views(host, 4, 3)
    assert b.ids.tolist() == [7, 8, 0, 0] and b.slot.tolist() == [1, 0, -1, -1] and b.entry.tolist() == [100, 200, -1, -1]
    assert b.block_table.view(4, 3).tolist() == [[5, 6, 0], [7, 0, 0], [0, 0, 0], [0, 0, 0]]
    assert b.cu.tolist() == [0, 1, 2, 3, 4] and all(sl.start % 4 == 0 for sl in lay.values())


# ------------------------------------------------------------------ scheduling
class _FakeRunner(HybridRunner):
    """The runner's bookkeeping with a model that answers (last token + 1) mod vocab."""

    def __init__(self, model, cache):
        super().__init__(model, cache)
        self.batches = []

    def step(self, entries):
        self.batches.append([len(t) for _, t, _ in entries])
        out = []
        for s, toks, want in entries:
            self.cache.reserve(s, len(toks))
            for w in want:
                row = torch.zeros(self.model.config.vocab_size)
                row[(toks[w] + 1) % row.numel()] = 1
                out.append(row)
        return torch.stack(out) if out else torch.zeros(0, self.model.config.vocab_size)

    def decode(self, seq_ids, last_tokens):
        return self.step([(s, [t], (0,)) for s, t in zip(seq_ids, last_tokens)])


def test_engine_packs_unequal_prompts_and_frees_everything():
    model = make_model(ODD, make_weights(ODD))
    runner = _FakeRunner(model, model.init_cache(3, num_blocks=12, block_size=8))
    eng = LLMEngine(model, runner=runner, max_batch_size=3)
    assert eng.cache is runner.cache
    prompts = [[1] * 5, [2] * 9, [3] * 2, [4] * 30, [5]]
    outs = eng.generate(prompts, SamplingParams(max_new_tokens=4))
    assert outs == [[p[0] + 1 + i for i in range(4)] for p in prompts]
    assert runner.batches[0] == [5, 9, 2]            # three requests of different lengths in one pass
    assert max(len(b) for b in runner.batches) == 3
    assert runner.cache.pool.num_free == 12 and len(runner.cache.free_slots) == 3


def test_long_prompts_run_in_portions():
    model = make_model(ODD, make_weights(ODD))
    runner = _FakeRunner(model, model.init_cache(1))
    runner.max_portion = 16
    runner.cache.add_sequence(0)
    runner.prefill(0, list(range(50)), 0)
    assert runner.batches == [[16], [16], [16], [2]] and runner.cache.lens[0] == 50


def test_engine_refuses_what_the_pool_cannot_hold():
    model = make_model(ODD, make_weights(ODD))
    eng = LLMEngine(model, runner=_FakeRunner(model, model.init_cache(2, num_blocks=2, block_size=4)), max_batch_size=2)
    rid = eng.submit([1] * 50, SamplingParams(max_new_tokens=2))
    ok = eng.submit([1] * 3, SamplingParams(max_new_tokens=2))
    eng.run_until_done()
    assert rid in eng.failed and eng.finished[ok].output == [2, 3]


# ------------------------------------------------------------------ the oracle's own properties
def test_oracle_recurrences_can_be_cut_anywhere():
    g = torch.Generator().manual_seed(1)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)  # noqa: E731
    q, k, v, f, beta = r(9, 2, 3), oracle.unit(r(9, 2, 3)), r(9, 2, 4), torch.sigmoid(r(9, 2, 3)), torch.sigmoid(r(9, 2))
    for fn, args in ((oracle.gated_write, (q, f, v)), (oracle.delta_rule, (q, k, v, beta, f))):
        whole, S = fn(*args)
        a, Sa = fn(*[x[:4] for x in args])
        b, Sb = fn(*[x[4:] for x in args], S=Sa)
        assert torch.allclose(torch.cat([a, b]), whole) and torch.allclose(Sb, S)


def test_oracle_chunk_and_rotation():
    assert oracle.chunk_visible(5, 5, 4) and oracle.chunk_visible(5, 4, 4) and not oracle.chunk_visible(5, 3, 4)
    assert not oracle.chunk_visible(4, 5, 4)
    x = torch.randn(3, 2, 6, dtype=torch.float64)
    y = oracle.rotate(x, 4, 100.0)
    assert torch.allclose(y[0], x[0]) and torch.allclose(y[..., 4:], x[..., 4:])
    assert torch.allclose((y[..., :2] ** 2).sum(-1), (x[..., :2] ** 2).sum(-1))
    assert torch.allclose(oracle.rotate(x[1:], 4, 100.0, start=1), y[1:])
    u = torch.arange(4.0).view(4, 1)
    assert oracle.short_conv(u, torch.tensor([[10.0, 1.0]])).flatten().tolist() == [0, 1, 12, 23]
    assert np.isclose(float(oracle.xielu(torch.tensor(0.0), torch.tensor(1.0), torch.tensor(1.0))), 0)
    assert attn(1, 1, 2, 2, 1, 3, 2, 1.0) and delta(1, 1, 2, 2, 1) and hgrn2(1, 2, 3) and parallel({}, {}, 1, 1)["mlp"] is None
