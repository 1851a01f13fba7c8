"""Rilenex kernels, cache and serving path on a B200 against the plain oracle (float64, no shared code)."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import rilenex_oracle as oracle
from rilenex_common import CONFIGS, ODD, TENSOR, attn, config, delta, hgrn2, make_model, make_weights, parallel

pytestmark = pytest.mark.gpu

if torch.cuda.is_available():
    from sneppx_alg_b200.hub.formats import save_safetensors
    from sneppx_alg_b200.nn.mixers import DeltaBranch, FusedMixer, GatedWriteBranch, TalkingAttentionBranch  # noqa: F401
    from sneppx_alg_b200.ops import check_status, hybrid
    from sneppx_alg_b200.ops.gemm import XIELU, gemm
    from sneppx_alg_b200.ops.ragged import RaggedBatch
    from sneppx_alg_b200.serving.generation import generate
    from sneppx_alg_b200.serving.hybrid_runner import HybridRunner
    from sneppx_alg_b200.serving.kv_cache import ChunkedKVCache
    from sneppx_alg_b200.serving.llm_engine import LLMEngine, SamplingParams

F32, BF16 = torch.float32, torch.bfloat16
TOL = {F32: 2e-4, BF16: 6e-2}      # rms of the logits' error over their rms; bf16: whole-model rounding
_cache = {}


def toks(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def model_of(name, dtype):
    if (name, dtype) not in _cache:
        W = make_weights(CONFIGS[name])
        _cache[name, dtype] = (make_model(CONFIGS[name], W, dtype, "cuda"), W)
    return _cache[name, dtype]


def want_logits(name, tokens):
    key = (name, tuple(tokens))
    if key not in _cache:
        _cache[key] = oracle.forward(CONFIGS[name], make_weights(CONFIGS[name]), tokens)
    return _cache[key]


def new_runner(model, n=4, poison=True, graphs=False, blocks=None, block_size=16):
    """A runner whose whole memory holds NaN: nothing may be read that the sequence has not written."""
    r = HybridRunner(model, model.init_cache(n, blocks, block_size))
    if poison:
        for t in r.cache.k + r.cache.v + [t for s in r.cache.state for t in s.values()]:
            t.fill_(float("nan"))
    if graphs:
        r.enable_graphs(n)
    return r


def close(got, want, dtype, tol=None):
    got, want = got.double().cpu(), want.double().cpu()
    assert got.shape == want.shape and torch.isfinite(got).all()
    err = ((got - want) ** 2).mean(-1).sqrt() / want.std()
    assert float(err.max()) < (tol or TOL[dtype]), float(err.max())


def feed(runner, seq, tokens, cuts):
    """Logits of every position with the tokens cut into portions at ``cuts``."""
    out, bounds = [], [0, *cuts, len(tokens)]
    for a, b in zip(bounds, bounds[1:]):
        out.append(runner.step([(seq, tokens[a:b], range(b - a))]))
    return torch.cat(out)


# ------------------------------------------------------------------ single mechanisms
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("width", [40, 72, 101, 4100])
def test_fp32_residual_norm_and_embedding(dtype, width):
    table = torch.randn(50, width, device="cuda").to(dtype)
    ids = torch.tensor([3, 49, 0, 7], dtype=torch.int32, device="cuda")
    x = hybrid.embed_f32(table, ids)
    assert torch.equal(x, table[ids.long()].float())
    w, rows = 1 + torch.rand(width, device="cuda"), torch.tensor([2, 0], dtype=torch.int32, device="cuda")
    x = x * 100
    want = oracle.rms(x.double(), 1e-3, w.double())
    atol = 1e-5 if dtype == F32 else 2e-2
    assert torch.allclose(hybrid.rmsnorm_f32(x, w, 1e-3, dtype).double(), want, atol=atol, rtol=atol)
    assert torch.allclose(hybrid.rmsnorm_f32(x, w, 1e-3, dtype, rows=rows).double(), want[[2, 0]], atol=atol, rtol=atol)


@pytest.mark.parametrize("rows", [3, 64, 300])
def test_xielu_and_fp32_residual_in_gemm_epilogues(rows):
    x, w = torch.randn(rows, 512, device="cuda").bfloat16(), (torch.randn(320, 512, device="cuda") / 20).bfloat16()
    act = XIELU(0.4, -0.9)
    z = x.double() @ w.double().T
    p, q = torch.tensor(0.4).double().cuda(), torch.tensor(-0.9).double().cuda()
    assert torch.allclose(gemm(x, w, act=act, out_dtype=F32).double(), oracle.xielu(z, p, q), atol=2e-3, rtol=1e-3)
    res = torch.randn(rows, 320, device="cuda")
    keep = res.clone()
    gemm(x, w, c=res, beta=1.0, out=res)
    assert torch.allclose(res.double(), keep.double() + z, atol=2e-3)


def one_layer(spec, seed=3, width=64, vocab=33):
    cfg = config(width, vocab, [spec], eps=1e-4)
    return cfg, make_weights(cfg, seed)


# left only, right only (scale of the other branch 0), recurrence alone; sizes on and off the tensor-core paths
SINGLES = {
    "hgrn2 small": hgrn2(2, 12, 7), "hgrn2 one head": hgrn2(1, 33, 5), "hgrn2 wide": hgrn2(2, 200, 24), "hgrn2 128": hgrn2(3, 128, 80),
    "delta grouped": parallel(attn(1, 1, 2, 8, 1, 4, 2, 1.0), delta(6, 3, 16, 24, 4), 0.0, 1.0),
    "delta odd": parallel(attn(1, 1, 2, 8, 1, 4, 2, 1.0), delta(5, 1, 27, 9, 7), 0.0, -0.7),
    "delta 128": parallel(attn(1, 1, 2, 8, 1, 4, 2, 1.0), delta(2, 2, 128, 64, 2), 0.0, 1.0),
    "delta no conv": parallel(attn(1, 1, 2, 8, 1, 4, 2, 1.0), delta(2, 1, 250, 16, 1), 0.0, 1.0),
    "attention one head": parallel(attn(1, 1, 16, 8, 3, 20, 16, 0.6), delta(1, 1, 4, 4, 1), 1.0, 0.0),
    "attention no rotation": parallel(attn(4, 2, 20, 12, 2, 33, 0, 0.5), delta(1, 1, 4, 4, 1), -1.2, 0.0),
    "attention grouped": parallel(attn(12, 3, 64, 128, 4, 50, 48, 0.3, 5e5), delta(1, 1, 4, 4, 1), 1.0, 0.0),
    "attention wide": parallel(attn(10, 10, 64, 16, 1, 64, 64, 0.2), delta(1, 1, 4, 4, 1), 1.0, 0.0),
    "attention large values": parallel(attn(4, 2, 32, 160, 6, 29, 32, 0.4), delta(1, 1, 4, 4, 1), 1.0, 0.0),
    "attention 20 heads": parallel(attn(20, 1, 16, 24, 2, 1000, 8, 0.4), delta(1, 1, 4, 4, 1), 1.0, 0.0),
}


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(SINGLES))
def test_one_mixer(name, dtype):
    cfg, W = one_layer(SINGLES[name])
    model = make_model(cfg, W, dtype, "cuda")
    t = toks(75, cfg["vocab"])
    layers = []
    want = oracle.forward(cfg, W, t, layers_out=layers)
    seen = []
    model.layers[0].register_forward_hook(lambda m, a, o: seen.append(a[0].clone()))
    r = new_runner(model)
    r.cache.add_sequence(0)
    got = feed(r, 0, t, [40, 41, 43] + list(range(64, 75)))
    close(got, want, dtype)
    # the branch itself, not hidden behind the residual stream
    x0 = W["embed"][t].double()
    got_x, want_x = torch.cat(seen).double().cpu() - x0, layers[0] - x0
    err = ((got_x - want_x) ** 2).mean(-1).sqrt() / want_x.std()
    assert float(err.max()) < (1e-4 if dtype == F32 else 5e-2), float(err.max())
    check_status()


def test_rotation_at_far_positions():
    """Angles stay exact where p * f in 32-bit would not."""
    d, rot, base, H = 8, 6, 1e4, 2
    inv = base ** (-2.0 * torch.arange(rot // 2, dtype=torch.float64) / rot)
    u = torch.randn(1, H * d + 2 * d, device="cuda")
    ring, one = torch.zeros(1, 1, H * d + 2 * d, device="cuda"), torch.ones(1, H * d + 2 * d, device="cuda")
    cache, w = torch.zeros(1, 16, 1, d, device="cuda"), 1 + torch.rand(d, device="cuda")
    for pos in (0, 1, 4095, 1_000_003):
        buf = torch.zeros(RaggedBatch.decode_layout(1, 1)[1], dtype=torch.int32)
        RaggedBatch.fill_decode(buf.numpy(), 1, 1, [0], [pos], [0], [3], [[0]], [pos // 16])
        b = RaggedBatch.decode_views(buf.cuda(), 1, 1)
        q = torch.empty(1, H, d, device="cuda")
        hybrid.qkv_prep(u, one, ring, w, w, inv.cuda(), b, cache, torch.zeros_like(cache), H, 1, d, d, 1, 1e-6, q_out=q)
        want = oracle.rotate(oracle.rms(u.cpu().double()[:, :H * d].view(1, H, d), 1e-6, w.cpu().double()), rot, base, start=pos)
        assert torch.allclose(q.cpu().double(), want, atol=2e-6), pos
        k = oracle.rotate(oracle.rms(u.cpu().double()[:, H * d:H * d + d].view(1, 1, d), 1e-6, w.cpu().double()), rot, base, start=pos)
        assert torch.allclose(cache[0, 3].cpu().double(), k[0], atol=2e-6)


# ------------------------------------------------------------------ visibility of single keys
KERNELS = ["simt prompt f32", "simt prompt bf16", "tensor prompt", "simt decode f32", "simt decode bf16", "tensor decode"]


def attend(kernel, q, k, v, talk, size, queries, bs=8, H=4, G=2):
    """Outputs of one sequence for the listed query positions with every attention kernel; gate closed to factor 1 / 2."""
    T, d, dv = q.shape[0], q.shape[2], v.shape[2]
    dt = F32 if "f32" in kernel else BF16
    kd, vd, t = k.to(dt).cuda(), v.to(dt).cuda(), talk.float().cuda()
    qmix = torch.einsum("hjg,tjgd->thjd", talk.view(H, G, H // G), q.view(T, G, H // G, d)).reshape(T, H, G * d)
    pad = torch.zeros(T, H, (G * d + 63) // 64 * 64)
    pad[..., :G * d] = qmix
    out = []
    for i in queries:
        y = torch.empty(1, H * dv, dtype=dt, device="cuda")
        gate = torch.zeros(1, 8, dtype=dt, device="cuda")
        if "prompt" in kernel:
            first = i // size * size
            lo = min(i, first + 3) if first + 3 < i else i       # portion [lo, i]: earlier chunk keys are carried rows
            n = i - lo + 1
            b = RaggedBatch.prompt("cuda", [[0] * n], [lo], [0], [[-1] * n], {size: [[0] * (lo - first)]}, [0])
            view = b.views[size]
            kk, vv = kd[first:i + 1].reshape(-1, G * d).contiguous(), vd[first:i + 1].reshape(-1, G * dv).contiguous()
            assert view.rows == kk.shape[0]
            yy, gg = y.expand(n, -1).contiguous(), gate.expand(n, -1).contiguous()
            if kernel.startswith("simt"):
                hybrid.talking_attention(q[lo:i + 1].float().contiguous().cuda(), kk, vv, t, gg, yy, b, view.kv_base, 1.0, 2.0, H, G, d, dv, dv, size)
            else:
                assert hybrid.talking_tc(dt, H, G, d, dv)
                hybrid.talking_attention_tc(pad[lo:i + 1].to(dt).contiguous().cuda(), kk, vv, gg, yy, b, view, 1.0, 2.0, H, G, d, dv, dv, size)
            y = yy[-1:]
        else:
            cache = ChunkedKVCache([(G, d, dv)], [size], 64, bs, dtype=dt, device="cuda")
            cache.k[0].fill_(float("nan"))
            cache.v[0].fill_(float("nan"))
            cache.add_sequence(0)
            for p in range(i + 1):
                e = cache.reserve(0, 1)[0]
                cache.k[0].view(-1, G, d)[e], cache.v[0].view(-1, G, dv)[e] = kd[p], vd[p]
            w = cache.table_width
            buf = torch.zeros(RaggedBatch.decode_layout(1, w)[1], dtype=torch.int32)
            RaggedBatch.fill_decode(buf.numpy(), 1, w, [0], [i], [0], [0], [cache.tables[0]], [cache.base[0]])
            b = RaggedBatch.decode_views(buf.cuda(), 1, w)
            tc = kernel.startswith("tensor")
            assert not tc or hybrid.talking_decode_tc(dt, H, G, d, dv)
            hybrid.talking_decode(None if tc else q[i:i + 1].float().contiguous().cuda(), cache.k[0], cache.v[0], t, gate, y, b, 1.0, 2.0, H, G, d, dv,
                                  size, qmix=pad[i:i + 1].to(dt).contiguous().cuda() if tc else None)
        out.append(y.float().cpu().view(H, dv))
    check_status()
    return torch.stack(out)


@pytest.mark.parametrize("kernel", KERNELS)
@pytest.mark.parametrize("size", [5, 24, 130, 300])
def test_a_key_that_stands_out_is_seen_exactly_inside_its_chunk(kernel, size):
    H, G, d, dv, T = 4, 2, 16, 16, 310
    g = torch.Generator().manual_seed(size)
    q, k, v = torch.randn(T, H, d, generator=g) * 0.1, torch.randn(T, G, d, generator=g) * 0.1, torch.randn(T, G, dv, generator=g) * 0.1
    talk = torch.eye(H) + 0.1 * torch.rand(H, H, generator=g)
    q[..., 0] = 4.0
    edge = size if size < 200 else 300
    spots = sorted({0, 1, 7, 8, edge - 1, edge, edge + 1, max(0, edge - 9), 127, 128})      # first tokens, block and chunk edges
    for spot in spots:
        kk, vv = k.clone(), v.clone()
        kk[spot, :, 0] = 8.0                       # score 32 above the rest: its weight is 1 wherever it is visible
        vv[spot] = 5.0
        queries = sorted({i for i in (spot - 1, spot, spot + 1, spot // size * size + size - 1, spot // size * size + size, 309) if 0 <= i < T})
        got = attend(kernel, q, kk, vv, talk, size, queries)
        for i, y in zip(queries, got):
            seen = oracle.chunk_visible(i, spot, size)
            assert (y > 4.9).all() if seen else (y < 1.0).all(), (spot, i, seen)


@pytest.mark.parametrize("kernel", KERNELS)
def test_attention_kernels_against_the_oracle(kernel):
    H, G, d, dv, T, size = 6, 2, 24, 40, 150, 64
    g = torch.Generator().manual_seed(5)
    q, k, v = (torch.randn(T, n, w, generator=g).bfloat16().float() for n, w in ((H, d), (G, d), (G, dv)))
    talk = torch.eye(H) * 0.7 + 0.3 * torch.randn(H, H, generator=g)
    want = oracle.talking_attention(q.double(), k.double(), v.double(), 1.0, talk.double(), size)
    queries = [0, 1, 31, 62, 63, 64, 100, 127, 128, 149]
    got = attend(kernel, q, k, v, talk, size, queries, bs=16, H=H, G=G)
    assert torch.allclose(got.double(), want[queries], atol=2e-5 if "f32" in kernel else 4e-2)


# ------------------------------------------------------------------ whole models: prompts, portions, decoding
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompt_decode_and_portions(name, dtype):
    model, _ = model_of(name, dtype)
    t = toks(101, CONFIGS[name]["vocab"])
    want = want_logits(name, t)
    for cuts in ([], [1], [2, 4], [16, 32, 33], [23, 24, 25, 48], [99], list(range(2, 101, 2)), list(range(1, 101)),
                 [47, 48, 49, 50, 66], [7, 21, 60]):
        r = new_runner(model, graphs=len(cuts) == 100)
        r.cache.add_sequence(5)
        close(feed(r, 5, t, cuts), want, dtype)
    check_status()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_first_tokens(name, dtype):
    model, _ = model_of(name, dtype)
    for n in (1, 2, 3, 4):
        t = toks(n, CONFIGS[name]["vocab"], seed=n)
        r = new_runner(model)
        r.cache.add_sequence(0)
        close(feed(r, 0, t, []), want_logits(name, t), dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_layers_one_by_one(dtype):
    model, W = model_of("tensor", dtype)
    t, want = toks(60, TENSOR["vocab"]), []
    oracle.forward(TENSOR, W, t, layers_out=want)
    seen, hooks = [], []
    for layer in model.layers:
        hooks.append(layer.register_forward_hook(lambda m, a, o: seen.append(a[0].clone())))
    r = new_runner(model)
    r.cache.add_sequence(0)
    r.step([(0, t, ())])
    for h in hooks:
        h.remove()
    assert len(seen) == len(want)
    for a, b in zip(seen, want):
        close(a, b, dtype, 1e-5 if dtype == F32 else 3e-2)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_unequal_requests_in_one_batch(name, dtype):
    model, _ = model_of(name, dtype)
    lens, extra = [70, 1, 25, 48], [6, 3, 9, 1]
    seqs = [toks(n + e, CONFIGS[name]["vocab"], seed=10 + i) for i, (n, e) in enumerate(zip(lens, extra))]
    want = [want_logits(name, s) for s in seqs]
    r = new_runner(model, graphs=True)
    for i in range(4):
        r.cache.add_sequence(i)
    out = r.step([(i, seqs[i][:n], (0, n - 1)) for i, n in enumerate(lens)])
    close(out, torch.cat([want[i][[0, n - 1]] for i, n in enumerate(lens)]), dtype)
    done = list(lens)
    for step in range(max(extra)):
        live = [i for i in range(4) if done[i] < len(seqs[i])]
        out = r.step([(i, [seqs[i][done[i]]], (0,)) for i in live])
        close(out, torch.stack([want[i][done[i]] for i in live]), dtype)
        for i in live:
            done[i] += 1
            if done[i] == len(seqs[i]):
                r.cache.free_sequence(i)
    assert r.cache.pool.num_free == r.cache.pool.num_blocks
    check_status()


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_mixed_batch_of_portions_and_single_tokens(dtype):
    """A prompt's next portion beside decoding sequences; one waits."""
    model, _ = model_of("odd", dtype)
    seqs = [toks(80, ODD["vocab"], seed=20 + i) for i in range(3)]
    want = [want_logits("odd", s) for s in seqs]
    r, pos = new_runner(model), [0, 0, 0]
    for i in range(3):
        r.cache.add_sequence(i)
    for part in ([30, 5, 17], [1, 20, 0], [1, 2, 31], [25, 1, 1], [1, 1, 1], [2, 0, 3]):
        entries = [(i, seqs[i][pos[i]:pos[i] + n], range(n)) for i, n in enumerate(part) if n]
        out = r.step(entries)
        close(out, torch.cat([want[i][pos[i]:pos[i] + n] for i, n in enumerate(part) if n]), dtype)
        pos = [p + n for p, n in zip(pos, part)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_slots_and_blocks_used_again(name, dtype):
    """A small pool: sequences come and go, blocks that fall behind one sequence's chunk serve another in the same step."""
    model, _ = model_of(name, dtype)
    vocab, sizes = CONFIGS[name]["vocab"], model.init_cache(1).sizes
    blocks = 2 * ((max(sizes) + 6) // 8 + 1)
    r = new_runner(model, n=2, blocks=blocks, block_size=8, graphs=True)
    live, nxt = {}, 0
    for rnd in range(12):
        while len(live) < 2:
            s = toks([60, 9, 33, 50, 3, 71][nxt % 6], vocab, seed=40 + nxt % 6)
            r.cache.add_sequence(nxt)
            live[nxt] = [s, 0, want_logits(name, s)]
            nxt += 1
        n = [1, 13, 2, 40][rnd % 4]
        entries, want = [], []
        for i, (s, p, w) in live.items():
            part = s[p:p + n]
            entries.append((i, part, range(len(part))))
            want.append(w[p:p + n])
        close(r.step(entries), torch.cat(want), dtype)
        for i, part, _ in entries:
            live[i][1] += len(part)
            if live[i][1] == len(live[i][0]):
                r.cache.free_sequence(i)
                del live[i]
    check_status()


@pytest.mark.parametrize("dtype,name", [(F32, "odd"), (BF16, "tensor"), (F32, "tensor")])
def test_long_decoding(name, dtype):
    model, _ = model_of(name, dtype)
    t = toks(260, CONFIGS[name]["vocab"], seed=9)
    r = new_runner(model, n=1, graphs=True)
    r.cache.add_sequence(0)
    close(feed(r, 0, t, list(range(3, 260))), want_logits(name, t), dtype)
    assert len(r.cache.tables[0]) <= r.cache.table_width


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_model_of_recurrent_layers_only(dtype):
    cfg = config(56, 70, [hgrn2(2, 24, 16, 48), hgrn2(4, 16, 10, None)])
    W = make_weights(cfg, 4)
    model = make_model(cfg, W, dtype, "cuda")
    seqs = [toks(n, 70, seed=n) for n in (45, 20)]
    want = [oracle.forward(cfg, W, s) for s in seqs]
    r = new_runner(model, n=2, graphs=True)
    for i in range(2):
        r.cache.add_sequence(i)
    close(r.step([(i, seqs[i][:17], range(17)) for i in range(2)]), torch.cat([w[:17] for w in want]), dtype)
    for k in range(17, 20):
        close(r.step([(i, [seqs[i][k]], (0,)) for i in range(2)]), torch.stack([w[k] for w in want]), dtype)
    prompt = seqs[1][:5]
    eng = LLMEngine(model, max_batch_size=2)
    got = eng.generate([prompt, prompt], SamplingParams(max_new_tokens=4))
    assert got[0] == got[1] and (dtype == BF16 or got[0] == greedy(cfg, W, prompt, 4))


def test_results_do_not_depend_on_company_or_place():
    """Same sequence alone, in a batch, in another slot and other blocks: differences are rounding only."""
    model, _ = model_of("tensor", F32)
    a, b = toks(90, TENSOR["vocab"], seed=1), toks(77, TENSOR["vocab"], seed=2)
    r = new_runner(model)
    r.cache.add_sequence(0)
    alone = r.step([(0, a, range(90))])
    r = new_runner(model)
    for i in (7, 8):
        r.cache.add_sequence(i)
    both = r.step([(7, b, ()), (8, a, range(90))])
    assert float((alone - both).abs().max()) < 1e-4 * float(alone.std())


# ------------------------------------------------------------------ entry points
def greedy(cfg, W, prompt, n):
    t = list(prompt)
    for _ in range(n):
        t.append(int(oracle.forward(cfg, W, t)[-1].argmax()))
    return t[len(prompt):]


def test_greedy_generation_through_the_engine():
    model, W = model_of("odd", F32)
    prompts = [toks(n, ODD["vocab"], seed=60 + n) for n in (21, 1, 34, 8)]
    want = [greedy(ODD, W, p, 6) for p in prompts]
    for batch, graphs in ((4, True), (2, False)):
        eng = LLMEngine(model, num_blocks=40, block_size=8, max_batch_size=batch, cuda_graphs=graphs)
        assert isinstance(eng.runner, HybridRunner)
        assert eng.generate(prompts, SamplingParams(max_new_tokens=6)) == want
        assert eng.cache.pool.num_free == 40
    ids = torch.tensor([prompts[0]], device="cuda")
    assert generate(model, ids, 6)[0, 21:].tolist() == want[0]
    assert eng.generate([prompts[0]], SamplingParams(max_new_tokens=6, do_sample=True, top_k=1)) == [want[0]]
    loss = model(ids, labels=ids)["loss"]
    lg = want_logits("odd", prompts[0])
    ref = torch.nn.functional.cross_entropy(lg[:-1], torch.tensor(prompts[0][1:]))
    assert abs(float(loss) - float(ref)) < 1e-3


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_runner(tmp_path, dtype):
    W = make_weights(ODD)
    (tmp_path / "config.json").write_text(json.dumps(ODD))
    save_safetensors(str(tmp_path / "model.safetensors"), {k: v.bfloat16() for k, v in W.items()})
    a, b = toks(40, ODD["vocab"], seed=1), toks(12, ODD["vocab"], seed=2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:38], "want": [0, 37]}, {"id": "b", "tokens": b[:11], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[38:39], "want": []}, {"id": "b", "tokens": b[11:], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[39:], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "a", "tokens": b, "want": [11]}], "end": ["a"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(tmp_path),
                        "--max-tokens", "64"], input="\n".join(map(json.dumps, steps)) + "\n", capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    assert not os.path.exists(tmp_path / "1.f32")
    wa, wb = want_logits("odd", a), want_logits("odd", b)
    for step, want in ((0, wa[[0, 37]]), (2, wa[39:]), (3, wb[11:])):
        got = np.fromfile(tmp_path / f"{step}.f32", dtype="<f4").reshape(-1, ODD["vocab"])
        close(torch.from_numpy(got), want, getattr(torch, dtype))


def test_sizes_that_no_kernel_takes_are_refused():
    cfg, W = one_layer(hgrn2(1, 300, 8))
    model = make_model(cfg, W, F32, "cuda")
    r = new_runner(model, n=1)
    r.cache.add_sequence(0)
    with pytest.raises(RuntimeError):
        r.step([(0, [1, 2, 3], (0,))])
    assert delta(1, 1, 1, 1, 1)
