"""Tibalorn on the host: configuration, weight reader, masks, blocks and averages, ragged batches, scheduling, and the plain
oracle against itself. The kernels are covered by ``test_gpu_tibalorn.py``."""
import json
import math
import random

import pytest
import torch

import tibalorn_oracle as oracle
from rilenex_common import ODD as RILENEX_ODD
from tibalorn_common import CONFIGS, ODD, attention, config, make_model, make_weights, mamba2, yarn
from sneppx_alg_b200.hub.formats import save_safetensors
from sneppx_alg_b200.hub.model_hub import ModelHub
from sneppx_alg_b200.models import ModelConfig, build_model, config_from_name, list_models
from sneppx_alg_b200.nn.mixers import rotary_frequencies
from sneppx_alg_b200.ops.gemm import SoftCap, gemm
from sneppx_alg_b200.ops.ragged import Chunk, PooledWindow, RaggedBatch, as_mask
from sneppx_alg_b200.serving.hybrid_runner import HybridRunner
from sneppx_alg_b200.serving.kv_cache import ChunkedKVCache
from sneppx_alg_b200.serving.llm_engine import LLMEngine, SamplingParams
from sneppx_alg_b200.serving.trace_runner import _cache_size


# ------------------------------------------------------------------ configuration and weights
@pytest.mark.parametrize("name", list(CONFIGS))
def test_config_reads_and_round_trips(name, tmp_path):
    c = CONFIGS[name]
    cfg = ModelConfig.from_dict(c)
    assert cfg.architecture == "tibalorn" and cfg.vocab_size == c["vocab"] and cfg.hidden_size == c["width"]
    assert cfg.layer_norm_eps == c["norm"]["eps"] and cfg.embedding_scale == c["embedding"]["scale"] and cfg.logit_softcap == c["logit_softcap"]
    assert cfg.num_hidden_layers == len(c["layers"]) == len(cfg.layer_specs) and cfg.tie_word_embeddings and not cfg.validate()
    cfg.to_json(str(tmp_path / "c.json"))
    assert ModelConfig.from_json(str(tmp_path / "c.json")) == cfg


@pytest.mark.parametrize("fmt", ["safetensors", "sneppx"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_weights_load_from_a_folder_and_save_back(tmp_path, fmt, name):
    W = make_weights(CONFIGS[name])
    (tmp_path / "config.json").write_text(json.dumps(CONFIGS[name]))
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


def test_reader_refuses_what_does_not_fit():
    W = make_weights(ODD)
    model = make_model(ODD, W)
    with pytest.raises(KeyError):
        model.load_reference_state_dict({k: v for k, v in W.items() if k != "l1.mix.sink"})
    with pytest.raises(ValueError):
        model.load_reference_state_dict({**W, "embed": W["embed"][:, :-1]})
    for layer in ({"type": "other", "mixer": {}, "mlp": None}, mamba2(3, 8, 4, 2, 4, 1), mamba2(3, 8, 4, 3, 4, 5),
                  attention(2, 1, 8, 7, 4, 2, 4, 1.0), attention(2, 1, 8, 8, 4, 2, 10, 1.0), attention(2, 1, 8, 8, 4, 0, 4, 1.0)):
        with pytest.raises(ValueError):
            build_model(ModelConfig.from_dict(config(16, 8, [layer])))
    with pytest.raises(RuntimeError):
        model(torch.zeros(1, 3, dtype=torch.long))      # the kernels are required


def test_presets():
    assert set(list_models()["tibalorn"]) == {"tiny", "1B", "7B"}
    cfg = config_from_name("tibalorn-tiny")
    assert sum(t.numel() for _, t in build_model(cfg).tensors()) == cfg.estimate_parameters()
    assert 0.8e9 < config_from_name("tibalorn-1b").estimate_parameters() < 1.3e9


# ------------------------------------------------------------------ activations and frequencies
def test_activations_match_their_definitions():
    x, w = torch.randn(5, 8) * 3, torch.randn(6, 8)
    z = (x @ w.T).double()
    assert torch.allclose(gemm(x, w, act="relu2").double(), oracle.squared_relu(z), atol=1e-4)
    assert torch.allclose(gemm(x, w, act=SoftCap(2.5)).double(), oracle.softcap(z, 2.5), atol=1e-6)
    assert float(oracle.softcap(z, 2.5).abs().max()) <= 2.5


@pytest.mark.parametrize("dims,base,scaling", [(8, 500.0, None), (16, 1e4, yarn(4.0, 64, 6.0, 1.0)), (64, 3e5, yarn(6.0, 4096, 24.0, 1.5)),
                                               (32, 1e4, yarn(16.0, 128, 64.0, 32.0)), (6, 1e4, yarn(2.0, 10 ** 9, 1e-3, 1e-4)), (0, 1e4, None)])
def test_rotary_frequencies(dims, base, scaling):
    f, mul = rotary_frequencies(dims, base, scaling)
    want, wmul = oracle.rotary_frequencies(dims, base, scaling)
    assert f.tolist() == pytest.approx(want, rel=1e-14) and mul == pytest.approx(wmul)
    if scaling:
        assert mul == pytest.approx(1 + math.log(scaling["factor"]) / 10)


# ------------------------------------------------------------------ masks, blocks, averages
def test_masks():
    w = PooledWindow(24, 5)
    for i in range(200):
        for j in range(200):
            if oracle.token_visible(i, j, 24):
                assert j >= w.first(i)
        assert w.blocks_seen(i) == sum(oracle.block_visible(i, b, 5, 24) for b in range(60))
        assert i - w.first(i) < w.span and w.first(i) <= i // 5 * 5 and w.first(i) <= w.first(i + 1)
    assert as_mask(7) == Chunk(7) and as_mask(w) is w and PooledWindow(4, 9).span == 9


@pytest.mark.parametrize("masks,bs", [((PooledWindow(24, 5),), 16), ((PooledWindow(7, 16), PooledWindow(40, 3)), 4),
                                      ((PooledWindow(5, 8), PooledWindow(20, 8), 33), 8), ((PooledWindow(1, 1),), 4)])
def test_cache_keeps_what_is_needed_and_an_entry_per_average(masks, bs):
    rng = random.Random(0)
    cache = ChunkedKVCache([(1, 2, 2)], masks, 400, bs, dtype=torch.float32, device="cpu")
    rules = [as_mask(m) for m in masks]
    store = {}
    for seq in range(3):
        cache.add_sequence(seq)
    for _ in range(150):
        seq = rng.randrange(3)
        n, p0 = rng.choice([1, 1, 1, 2, 3, 17, 90]), cache.lens[seq]
        for m in rules:         # what the portion's first token still needs is there, and so is every average
            for p, e in zip(range(m.first(p0), p0), cache.entries(seq, m.first(p0), p0)):
                assert store[e] == (seq, p)
            if m.pool:
                for b, e in enumerate(cache.average_entries(seq, m.pool, 0, p0 // m.pool)):
                    assert store[e] == (seq, m.pool, b)
        entries = cache.reserve(seq, n)
        last = p0 + n - 1
        for p, e in zip(range(p0, p0 + n), entries):
            assert (e >= 0) == (p >= min(m.first(last) for m in rules))
            if e >= 0:
                store[e] = (seq, p)
        for pool in cache.pools:
            b0, b1 = p0 // pool, (p0 + n) // pool
            for b, e in zip(range(b0, b1), cache.average_entries(seq, pool, b0, b1)):
                store[e] = (seq, pool, b)
        assert len(cache.tables[seq]) <= cache.table_width
        assert cache.blocks_held(seq) <= cache.blocks_for(cache.lens[seq])
        live = [b for t in [cache.tables, *cache.averages.values()] for x in t.values() for b in x]
        assert len(set(live)) == len(live) and len(live) + cache.pool.num_free == 400
        if cache.lens[seq] > 500:
            cache.free_sequence(seq)
            cache.add_sequence(seq)
    for seq in range(3):
        cache.free_sequence(seq)
    assert cache.pool.num_free == 400 and all(not t for t in cache.averages.values())


def test_init_cache_has_room_for_its_sequences():
    model = make_model(ODD, make_weights(ODD))
    cache = model.init_cache(2, max_tokens=300, block_size=4)
    for seq in (0, 1):
        cache.add_sequence(seq)
        for _ in range(300):
            cache.reserve(seq, 1)
    with pytest.raises(MemoryError):
        for _ in range(200):
            cache.reserve(0, 1)
    slots, blocks = _cache_size(model, 100)
    assert slots == 100
    cache = model.init_cache(slots, blocks)
    for seq in range(100):                   # one token each, then one sequence with all of them
        cache.add_sequence(seq)
        cache.reserve(seq, 1)
    for seq in range(100):
        cache.free_sequence(seq)
    cache.add_sequence(0)
    for _ in range(100):
        cache.reserve(0, 1)


# ------------------------------------------------------------------ ragged batches
def test_prompt_batch_layout_with_averages():
    w = PooledWindow(6, 4)
    b = RaggedBatch.prompt("cpu", [[5] * 9, [8], [9] * 3], [0, 30, 6], [3, 0, 1], [[1] * 9, [4], [7, 8, 9]],
                           {w: [[], [50, 51, 52, 53, 54], [60, 61, 62, 63, 64, 65]]}, [2], averages={w: [([], [20, 21]), ([70, 71, 72, 73, 74, 75, 76], []), ([80], [81])]})
    v = b.views[w]
    # rows: 0 1 | - | 2 .. 10     11 .. 17 | - | 18 .. 22 | 23     24 25 | 26 .. 31 | 32 33 34
    assert v.rows == 35 and v.pool_base.tolist() == [0, 11, 24]
    assert v.kv_row.tolist() == list(range(2, 11)) + [23] + [32, 33, 34] and v.kv_base.tolist() == [2, 23 - 30, 32 - 6]
    assert v.gather_entry.tolist() == [70, 71, 72, 73, 74, 75, 76, 50, 51, 52, 53, 54, 80, 60, 61, 62, 63, 64, 65]
    assert v.gather_row.tolist() == list(range(11, 18)) + list(range(18, 23)) + [24] + list(range(26, 32))
    assert v.n_pool == 3 and v.pool_src.tolist() == [2, 6, 30] and v.pool_row.tolist() == [0, 1, 25] and v.pool_entry.tolist() == [20, 21, 81]


def test_decode_batch_layout_with_averages():
    lay, n = RaggedBatch.decode_layout(3, 2, (4, 6), 4)
    host = torch.full((n,), 9, dtype=torch.int32)
    RaggedBatch.fill_decode(host.numpy(), 3, 2, [7, 8], [20, 31], [1, 0], [100, 200], [[5, 6], [7]], [1, 1],
                            {4: ([-1, 33], [[2], [3, 4]]), 6: ([12, -1], [[], [11, 10, 9, 8]])}, 4)
    b = RaggedBatch.decode_views(host, 3, 2, (4, 6), 4)
    assert b.pool_entry[4].tolist() == [-1, 33, -1] and b.pool_entry[6].tolist() == [12, -1, -1]
    assert b.pool_table[4].view(3, 4).tolist() == [[2, 0, 0, 0], [3, 4, 0, 0], [0] * 4]
    assert b.pool_table[6].view(3, 4)[1].tolist() == [11, 10, 9, 8] and b.block_table.view(3, 2).tolist() == [[5, 6], [7, 0], [0, 0]]
    assert all(sl.start % 4 == 0 for sl in lay.values())


# ------------------------------------------------------------------ scheduling
class _FakeRunner(HybridRunner):
    """The runner's bookkeeping with a model that answers (last token + 1) mod vocab."""

    def step(self, entries):
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


def test_engine_counts_averages_when_it_admits():
    """The pool is just large enough for two requests at their full length; a third waits and nothing runs out of blocks."""
    model = make_model(ODD, make_weights(ODD))
    each = model.init_cache(1, 64, block_size=4).blocks_for(80)
    runner = _FakeRunner(model, model.init_cache(3, num_blocks=2 * each, block_size=4))
    eng = LLMEngine(model, runner=runner, max_batch_size=3)
    prompts = [[1] * 30, [2] * 60, [3] * 75, [4] * 2]
    params = [SamplingParams(max_new_tokens=80 - len(p)) for p in prompts]
    ids = [eng.submit(p, q) for p, q in zip(prompts, params)]
    most = 0
    while eng.has_work():
        eng.step()
        most = max(most, len(eng.running))
    assert most == 2 and not eng.failed and [len(eng.finished[i].output) for i in ids] == [50, 20, 5, 78]
    assert runner.cache.pool.num_free == 2 * each
    rid = eng.submit([1] * 79, SamplingParams(max_new_tokens=1000))
    eng.run_until_done()
    assert rid in eng.failed


def test_other_hybrid_models_use_the_same_base():
    from rilenex_common import make_model as rilenex_model, make_weights as rilenex_weights
    from sneppx_alg_b200.models.hybrid import HybridDecoder
    a, b = rilenex_model(RILENEX_ODD, rilenex_weights(RILENEX_ODD)), make_model(ODD, make_weights(ODD))
    assert isinstance(a, HybridDecoder) and isinstance(b, HybridDecoder) and a.head is not None and b.head is None


# ------------------------------------------------------------------ the oracle's own properties
def test_oracle_recurrence_can_be_cut_anywhere_and_is_a_sum():
    g = torch.Generator().manual_seed(1)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)  # noqa: E731
    x, B, C, dt, al, D = r(9, 4, 3), r(9, 2, 5), r(9, 2, 5), torch.rand(9, 4, generator=g, dtype=torch.float64), r(4), r(4)
    whole, S = oracle.ssd(x, B, C, dt, al, D)
    a, Sa = oracle.ssd(x[:4], B[:4], C[:4], dt[:4], al, D)
    b, Sb = oracle.ssd(x[4:], B[4:], C[4:], dt[4:], al, D, S=Sa)
    assert torch.allclose(torch.cat([a, b]), whole) and torch.allclose(Sb, S)
    t, h = 7, 3              # closed form of one output
    y = D[h] * x[t, h]
    for s in range(t + 1):
        y = y + (C[t, 1] @ B[s, 1]) * torch.exp(-torch.exp(al[h]) * dt[s + 1:t + 1, h].sum()) * dt[s, h] * x[s, h]
    assert torch.allclose(whole[t, h], y)


def test_oracle_attention_edges_and_rotation():
    assert oracle.token_visible(5, 5, 3) and oracle.token_visible(5, 3, 3) and not oracle.token_visible(5, 2, 3) and not oracle.token_visible(4, 5, 3)
    assert oracle.block_visible(10, 1, 4, 3) and not oracle.block_visible(9, 1, 4, 3)
    x = torch.randn(3, 2, 6, dtype=torch.float64)
    f, _ = oracle.rotary_frequencies(4, 100.0)
    y = oracle.rotate_half(x, f)
    assert torch.allclose(y[0], x[0]) and torch.allclose(y[..., 4:], x[..., 4:])
    assert torch.allclose(oracle.rotate_half(y, f, sign=-1), x)
    assert torch.allclose(oracle.rotate_half(x[1:], f, start=1), y[1:])
    u = torch.arange(4.0).view(4, 1)
    assert oracle.short_conv(u, torch.tensor([[10.0, 1.0]]), torch.tensor([0.5])).flatten().tolist() == [0.5, 1.5, 12.5, 23.5]
    # a sink takes its share: with equal scores 0 and sink 0, two tokens leave 2 / 3 of the weight on the values
    z, one = torch.zeros(2, 1, 4, dtype=torch.float64), torch.ones(1, dtype=torch.float64)
    o = oracle.pooled_window_attention(z, z, torch.ones(2, 1, 2, dtype=torch.float64), 1.0, one, 0 * one, 8, 4)
    assert torch.allclose(o[1], torch.full((1, 2), 2 / 3, dtype=torch.float64))
