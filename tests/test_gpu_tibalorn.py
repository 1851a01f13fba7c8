"""Tibalorn kernels, cache and serving path on a B200 against the plain oracle (float64, no shared code)."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import tibalorn_oracle as oracle
from tibalorn_common import CONFIGS, ODD, TENSOR, attention, config, make_model, make_weights, mamba2, yarn

pytestmark = pytest.mark.gpu

if torch.cuda.is_available():
    from sneppx_alg_b200.hub.formats import save_safetensors
    from sneppx_alg_b200.ops import check_status, hybrid
    from sneppx_alg_b200.ops.gemm import SoftCap, gemm
    from sneppx_alg_b200.ops.ragged import PooledWindow, RaggedBatch
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


def new_runner(model, n=4, graphs=False, blocks=None, block_size=16):
    """A runner whose whole memory holds NaN: nothing may be read that the sequence has not written."""
    r = HybridRunner(model, model.init_cache(n, blocks, block_size, max_tokens=512))
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
def test_layer_norm_and_scaled_embedding(dtype, width):
    table = torch.randn(50, width, device="cuda").to(dtype)
    ids = torch.tensor([3, 49, 0, 7], dtype=torch.int32, device="cuda")
    x = hybrid.embed_f32(table, ids, 1.3)
    assert torch.equal(x, table[ids.long()].float() * 1.3)
    w, b, rows = 1 + torch.rand(width, device="cuda"), torch.randn(width, device="cuda"), torch.tensor([2, 0], dtype=torch.int32, device="cuda")
    x = 0.1 * x + 30          # a mean far above the deviations
    want = oracle.layer_norm(x.double(), w.double(), b.double(), 1e-3)
    atol = 2e-4 if dtype == F32 else 3e-2
    assert torch.allclose(hybrid.layernorm_f32(x, w, b, 1e-3, dtype).double(), want, atol=atol, rtol=1e-2 if dtype == BF16 else 1e-5)
    assert torch.allclose(hybrid.layernorm_f32(x, w, b, 1e-3, dtype, rows=rows).double(), want[[2, 0]], atol=atol, rtol=1e-2)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("width,parts,pad", [(96, 3, 8), (60, 5, 1), (4096, 1, 0), (16384, 2, 16), (4096, 64, 0)])
def test_norm_of_parts(dtype, width, parts, pad):
    buf = (torch.randn(5, width + pad, device="cuda") * torch.rand(5, width + pad, device="cuda") * 4).to(dtype)
    y, keep = buf[:, :width], buf.clone()
    w = 1 + torch.rand(width, device="cuda")
    want = oracle.group_rms(y.double().contiguous(), parts, 1e-2, w.double())
    hybrid.part_rmsnorm_(y, w, parts, 1e-2)
    assert torch.allclose(y.double(), want, atol=1e-5 if dtype == F32 else 1e-2, rtol=1e-5 if dtype == F32 else 1e-2)
    assert torch.equal(buf[:, width:], keep[:, width:])


@pytest.mark.parametrize("rows", [3, 64, 300])
def test_activations_in_gemm_epilogues(rows):
    x, w = torch.randn(rows, 512, device="cuda").bfloat16(), (torch.randn(320, 512, device="cuda") / 8).bfloat16()
    z = x.double() @ w.double().T
    assert torch.allclose(gemm(x, w, act="relu2", out_dtype=F32).double(), oracle.squared_relu(z), atol=1e-3, rtol=1e-3)
    for cap in (2.0, 30.0):
        got = gemm(x, w, act=SoftCap(cap), out_dtype=F32).double()
        assert torch.allclose(got, oracle.softcap(z, cap), atol=2e-4) and float(got.abs().max()) <= cap


# one mixer each; sizes on and off the tensor-core paths
SINGLES = {
    "mamba2 grouped": mamba2(6, 10, 20, 3, 4, 2), "mamba2 one head": mamba2(1, 5, 33, 1, 2, 1), "mamba2 no conv": mamba2(3, 16, 16, 1, 1, 3),
    "mamba2 128": mamba2(4, 64, 128, 1, 4, 1), "mamba2 wide values": mamba2(2, 200, 24, 2, 8, 4), "mamba2 wide state": mamba2(2, 64, 250, 1, 5, 2),
    "attention plain": attention(4, 4, 32, 32, 20, 4, 32, 0.4), "attention one head": attention(1, 1, 16, 8, 3, 20, 16, 0.6),
    "attention no rotation of keys": attention(4, 2, 20, 12, 33, 7, 0, 0.5), "attention blocks of one": attention(4, 2, 24, 24, 9, 1, 8, 0.5),
    "attention window of one": attention(4, 2, 24, 24, 1, 3, 8, 0.5), "attention yarn": attention(4, 1, 64, 40, 30, 6, 48, 0.3, 1e3, yarn(6.0, 50, 5.0, 1.0)),
    "attention large values": attention(4, 2, 32, 160, 29, 5, 32, 0.4), "attention odd keys": attention(6, 3, 27, 6, 17, 4, 10, 0.4),
    "attention 20 heads": attention(20, 1, 16, 24, 31, 8, 8, 0.4), "attention 256": attention(2, 1, 256, 128, 40, 16, 64, 0.1),
    "attention never full": attention(4, 2, 48, 32, 1000, 12, 16, 0.3),
}


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(SINGLES))
def test_one_mixer(name, dtype):
    cfg = config(64, 33, [SINGLES[name]], eps=1e-4)
    W = make_weights(cfg, 3)
    model = make_model(cfg, W, dtype, "cuda")
    t = toks(141, cfg["vocab"])
    layers, seen = [], []
    want = oracle.forward(cfg, W, t, layers_out=layers)
    model.layers[0].register_forward_hook(lambda m, a, o: seen.append(a[0].clone()))
    r = new_runner(model)
    r.cache.add_sequence(0)
    got = feed(r, 0, t, [70, 71, 73] + list(range(128, 141)))
    close(got, want, dtype)
    # the mixer itself, not hidden behind the residual stream
    x0 = W["embed"][t].double()
    got_x, want_x = torch.cat(seen).double().cpu() - x0, layers[0] - x0
    err = ((got_x - want_x) ** 2).mean(-1).sqrt() / want_x.std()
    assert float(err.max()) < (1e-4 if dtype == F32 else 5e-2), float(err.max())
    check_status()


@pytest.mark.parametrize("interleaved", [False, True])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_rotation_bias_and_temperature_at_far_positions(interleaved, dtype):
    """Angles stay exact where p * f in 32-bit would not."""
    d, dv, rot, H, G = 10, 6, 8, 2, 1
    freqs, mul = oracle.rotary_frequencies(rot, 1e4, yarn(4.0, 100, 9.0, 1.0))
    vfreqs, _ = oracle.rotary_frequencies(dv, 1e4)
    f64 = lambda x: torch.tensor(x, dtype=torch.float64, device="cuda")  # noqa: E731
    u = torch.randn(1, H * d + d + dv, device="cuda").to(dtype)
    bias, temp = torch.randn(u.shape[1], device="cuda"), torch.tensor([0.5, -2.0], device="cuda")

    def pairs(x, n, back=False):      # neighbours <-> halves
        if not interleaved:
            return x
        i = torch.arange(2 * n)
        perm = torch.cat([i.view(n, 2).T.reshape(-1), torch.arange(2 * n, x.shape[-1])])
        return x[..., torch.argsort(perm)] if back else x[..., perm]

    for pos in (0, 1, 4095, 1_000_003):
        kc, vc = torch.zeros(1, 16, G, d, dtype=dtype, device="cuda"), torch.zeros(1, 16, G, dv, dtype=dtype, device="cuda")
        buf = torch.zeros(RaggedBatch.decode_layout(1, 1)[1], dtype=torch.int32)
        RaggedBatch.fill_decode(buf.numpy(), 1, 1, [0], [pos], [0], [3], [[0]], [pos // 16])
        b = RaggedBatch.decode_views(buf.cuda(), 1, 1)
        q = torch.empty(1, H, d, device="cuda")
        turn = hybrid.win_prep(u, bias, f64(freqs), f64(vfreqs), mul, temp, b, kc, vc, H, G, d, dv, interleaved, q32=q)
        x = (u.double() + bias.double()).cpu()
        rot_of = lambda y, n, f, m=1.0: pairs(oracle.rotate_half(pairs(y, n), f, m, start=pos), n, True)  # noqa: E731
        atol = 3e-6 if dtype == F32 else 2e-2
        want = rot_of(x[:, :H * d].view(1, H, d), rot // 2, freqs, mul) * temp.double().cpu()[None, :, None]
        assert torch.allclose(q.cpu().double(), want, atol=3e-6), pos
        assert torch.allclose(kc[0, 3].cpu().double(), rot_of(x[:, H * d:H * d + d].view(1, 1, d), rot // 2, freqs, mul)[0], atol=atol)
        assert torch.allclose(vc[0, 3].cpu().double(), rot_of(x[:, H * d + d:].view(1, 1, dv), dv // 2, vfreqs)[0], atol=atol)
        a = pos * torch.tensor(vfreqs, dtype=torch.float64)
        assert torch.allclose(turn.cpu().double()[0], torch.stack([torch.cos(a), torch.sin(a)], -1), atol=2e-6)


@pytest.mark.parametrize("P,N,G", [(64, 128, 1), (48, 24, 2), (20, 250, 1), (136, 64, 4), (7, 3, 1)])
def test_recurrence_prompt_forms_and_steps_leave_the_same_state(P, N, G):
    """The tensor-core scan, the scan of 32-bit runs and single steps on the same rows, from the same bf16 projections."""
    H, taps, T = 4, 4, 150
    c = H * P + 2 * G * N
    g = torch.Generator().manual_seed(P)
    u = torch.randn(T, (H * P + c + H + 7) // 8 * 8, generator=g)[:, :H * P + c + H].bfloat16()
    wide = torch.zeros(T, (H * P + c + H + 7) // 8 * 8, dtype=BF16)
    wide[:, :u.shape[1]] = u
    conv, cb = torch.randn(c, taps, generator=g) * 0.4, torch.randn(c, generator=g) * 0.2
    dtb, al, D = torch.randn(H, generator=g) - 2, torch.randn(H, generator=g) * 0.5 - 1, torch.randn(H, generator=g)
    ud = u.double()
    xbc = oracle.silu(oracle.short_conv(ud[:, H * P:H * P + c], conv.double(), cb.double()))
    x, B, C = xbc[:, :H * P].view(T, H, P), xbc[:, H * P:H * P + G * N].view(T, G, N), xbc[:, H * P + G * N:].view(T, G, N)
    y, S = oracle.ssd(x, B, C, oracle.softplus(ud[:, H * P + c:] + dtb.double()), al.double(), D.double())
    y = y.reshape(T, -1) * oracle.silu(ud[:, :H * P])
    dev = lambda t: t.float().contiguous().cuda()  # noqa: E731
    ws = [dev(conv.T), dev(cb)], [dev(dtb), dev(al), dev(D)]
    for dtype, cuts, seg in ((BF16, [150], 512), (F32, [150], 512), (BF16, [64, 1, 2, 60, 23], 512), (F32, [1] * 20 + [130], 512),
                             (BF16, [1] * 150, 512), (BF16, [150], 64), (BF16, [2, 128, 20], 64), (BF16, [10, 140], 128)):
        ring, state = torch.full((2, taps, c), float("nan"), dtype=dtype, device="cuda"), torch.full((2, H, N, P), float("nan"), device="cuda")
        out, at = [], 0
        for n in cuts:
            rows = wide[at:at + n].to(dtype).cuda()[:, :u.shape[1]]
            o = torch.empty(n, (H * P + 7) // 8 * 8, dtype=dtype, device="cuda")[:, :H * P]
            if n == 1:
                buf = torch.zeros(RaggedBatch.decode_layout(1, 0)[1], dtype=torch.int32)
                RaggedBatch.fill_decode(buf.numpy(), 1, 0, [0], [at], [1], [-1], [[]], [0])
                hybrid.ssd_step(rows, *ws[0], ring, *ws[1], state, o, RaggedBatch.decode_views(buf.cuda(), 1, 0), H, P, N, G, taps)
            else:
                b = RaggedBatch.prompt("cuda", [[0] * n], [at], [1], [[-1] * n], {}, [0], segment_rows=seg)
                hybrid.ssd_prompt(rows, *ws[0], ring, *ws[1], state, o, b, H, P, N, G, taps)
            out.append(o.double().cpu())
            at += n
        tol = 2e-5 if dtype == F32 else 1.5e-2
        assert float((torch.cat(out) - y).abs().max()) < tol * float(y.abs().max())
        # bf16: x and B are rounded once where they enter; the state itself is fp32
        assert float((state[1].double().cpu() - S).abs().max()) < (1e-5 if dtype == F32 else 8e-3) * float(S.abs().max())
        assert torch.isnan(state[0]).all()
    check_status()


def test_segments_of_several_sequences_run_side_by_side():
    """Unequal portions, some of one segment, one that goes on from a stored state: the same as without segments."""
    H, P, N, G, taps = 2, 40, 24, 1, 3
    c = H * P + 2 * G * N
    lens, pos0 = [300, 64, 65, 1, 190], [0, 7, 0, 12, 90]
    g = torch.Generator().manual_seed(1)
    u = torch.randn(sum(lens), (H * P + c + H + 7) // 8 * 8, generator=g).bfloat16().cuda()[:, :H * P + c + H]
    w = [torch.randn(taps, c, generator=g).cuda() * 0.4, torch.randn(c, generator=g).cuda() * 0.2]
    v = [torch.randn(H, generator=g).cuda() - 2, torch.randn(H, generator=g).cuda() * 0.5 - 1, torch.randn(H, generator=g).cuda()]
    S0, R0 = torch.randn(5, H, N, P, generator=g), torch.randn(5, taps, c, generator=g).bfloat16()
    out = []
    for seg in (512, 64, 128):
        state, y = S0.cuda(), torch.empty(sum(lens), H * P, dtype=BF16, device="cuda")
        b = RaggedBatch.prompt("cuda", [[0] * n for n in lens], pos0, [4, 0, 2, 1, 3], [[-1] * n for n in lens], {}, [0], segment_rows=seg)
        hybrid.ssd_prompt(u, *w, R0.cuda(), *v, state, y, b, H, P, N, G, taps)
        out.append((y.double(), state.double()))
    assert b.n_segments == 3 + 1 + 1 + 1 + 2
    for y, state in out[1:]:
        assert torch.allclose(state, out[0][1], atol=2e-4, rtol=2e-4) and torch.allclose(y, out[0][0], atol=2e-2, rtol=2e-2)


# ------------------------------------------------------------------ visibility of single keys and blocks
KERNELS = ["simt prompt f32", "simt prompt bf16", "tensor prompt", "simt decode f32", "simt decode bf16", "tensor decode"]


def attend(kernel, q, k, v, sink, size, pool, queries, bs=8, H=4, G=2, interleaved=False):
    """Outputs of one sequence for the listed query positions with every attention kernel; rotation off, gate open by half."""
    T, d, dv = q.shape[0], q.shape[2], v.shape[2]
    dt, win = F32 if "f32" in kernel else BF16, PooledWindow(size, pool)
    kd, vd, sk = k.to(dt).cuda(), v.to(dt).cuda(), sink.float().cuda()
    nb = T // pool
    kb, vb = (x[:nb * pool].float().view(nb, pool, G, -1).mean(1).to(dt) for x in (kd, vd))
    tc = kernel.startswith("tensor")
    out = []
    for i in queries:
        if "prompt" in kernel:
            lo = max(0, i - 3) if i % 3 else i           # portion [lo, i]: earlier keys are carried rows
            n, first = i - lo + 1, win.first(lo)
            b0, b1 = lo // pool, (i + 1) // pool
            b = RaggedBatch.prompt("cuda", [[0] * n], [lo], [0], [[-1] * n], {win: [[0] * (lo - first)]}, [0],
                                   averages={win: [([0] * b0, [0] * (b1 - b0))]})
            view = b.views[win]
            kk = torch.cat([kb[:b1], kd[first:i + 1]]).reshape(-1, G * d).contiguous()
            vv = torch.cat([vb[:b1], vd[first:i + 1]]).reshape(-1, G * dv).contiguous()
            assert view.rows == kk.shape[0]
        else:
            cache = ChunkedKVCache([(G, d, dv)], [win], 400, bs, dtype=dt, device="cuda")
            cache.k[0].fill_(float("nan"))
            cache.v[0].fill_(float("nan"))
            cache.add_sequence(0)
            e = cache.reserve(0, i + 1)
            keep = [p for p in range(i + 1) if e[p] >= 0]
            e, a = [e[p] for p in keep], cache.average_entries(0, pool, 0, (i + 1) // pool)
            cache.k[0].view(-1, G, d)[e], cache.v[0].view(-1, G, dv)[e] = kd[keep], vd[keep]
            cache.k[0].view(-1, G, d)[a], cache.v[0].view(-1, G, dv)[a] = kb[:len(a)], vb[:len(a)]
            w, pw, n, lo = cache.table_width, 64, 1, i
            buf = torch.zeros(RaggedBatch.decode_layout(1, w, (pool,), pw)[1], dtype=torch.int32)
            RaggedBatch.fill_decode(buf.numpy(), 1, w, [0], [i], [0], [0], [cache.tables[0]], [cache.base[0]], {pool: ([-1], [cache.averages[pool][0]])}, pw)
            b = RaggedBatch.decode_views(buf.cuda(), 1, w, (pool,), pw)
        turn = torch.zeros(n, dv // 2, 2, device="cuda")
        turn[..., 0] = 1
        y, gate = torch.empty(n, H * dv, dtype=dt, device="cuda"), torch.zeros(n, H * dv, dtype=dt, device="cuda")
        if tc:
            up = 64 if "prompt" in kernel else 16
            qq = torch.zeros(n, H, (d + up - 1) // up * up, dtype=dt, device="cuda")
            qq[..., :d] = q[lo:i + 1]
            qa = dict(q=qq)
        else:
            qa = dict(q32=q[lo:i + 1].float().contiguous().cuda())
        if "prompt" in kernel:
            assert not tc or hybrid.window_tc(dt, H, G, d, dv)
            hybrid.window_attention(kk, vv, d, dv, sk, turn, gate, y, b, view, 1.0, H, G, d, dv, win, interleaved, **qa)
        else:
            assert not tc or hybrid.window_decode_tc(dt, H, G, d, dv)
            hybrid.window_decode(cache.k[0], cache.v[0], sk, turn, gate, y, b, 1.0, H, G, d, dv, win, interleaved, **qa)
        out.append(2 * y[-1].float().cpu().view(H, dv))
    check_status()
    return torch.stack(out).double()


@pytest.mark.parametrize("kernel", KERNELS)
@pytest.mark.parametrize("size,pool", [(5, 3), (24, 8), (130, 4), (300, 40), (3, 16)])
def test_a_key_that_stands_out_is_seen_as_token_then_not_then_in_its_block(kernel, size, pool):
    H, G, d, dv, T = 4, 2, 16, 16, 420
    g = torch.Generator().manual_seed(size)
    q, k, v = torch.randn(T, H, d, generator=g) * 0.1, torch.randn(T, G, d, generator=g) * 0.1, torch.randn(T, G, dv, generator=g) * 0.1
    q, k, v = (x.bfloat16().float() for x in (q, k, v))
    q[..., 0] = 4.0
    sink, one = torch.zeros(H), torch.ones(H, dtype=torch.float64)
    for spot in sorted({0, 1, 7, 8, pool - 1, pool, 2 * pool + 1, 63, 64, 127, 128}):
        kk, vv = k.clone(), v.clone()
        kk[spot, :, 0] = 8.0 * pool            # also the block's average has a score far above the rest
        vv[spot] = 64.0
        end = spot // pool * pool + pool - 1   # last position of its block
        at = sorted({i for i in (spot - 1, spot, spot + 1, spot + size - 1, spot + size, end + size - 1, end + size, end + size + 1, T - 1)
                     if 0 <= i < T})
        want = oracle.pooled_window_attention(q.double(), kk.double(), vv.double(), 1.0, one, sink.double(), size, pool, at=at)[at]
        got = attend(kernel, q, kk, vv, sink, size, pool, at)
        assert torch.allclose(got, want, atol=0.05, rtol=0.02), (spot, [(i, float(a.mean()), float(b.mean())) for i, a, b in zip(at, got, want)])
        for i, w in zip(at, want):             # the test's own premise: each state can be told from the others
            seen = oracle.token_visible(i, spot, size), oracle.block_visible(i, spot // pool, pool, size)
            assert not all(seen) and (w > 60).all() == seen[0] or pool == 1
            assert seen[0] or ((w.abs() > 0.9 * 64 / pool).all() == seen[1] or pool > 16)


@pytest.mark.parametrize("kernel", KERNELS)
@pytest.mark.parametrize("interleaved", [False, True])
def test_attention_kernels_against_the_oracle(kernel, interleaved):
    """A sink above all scores, one below, a score range that forces rescaling; pairs are not turned here, so their layout does
    not matter."""
    H, G, d, dv, T, size, pool = 6, 2, 24, 40, 300, 64, 7
    g = torch.Generator().manual_seed(5)
    q, k, v = (torch.randn(T, n, w, generator=g).bfloat16().float() for n, w in ((H, d), (G, d), (G, dv)))
    k = (k * torch.linspace(0.2, 2.0, T)[:, None, None]).bfloat16().float()
    sink = torch.tensor([20.0, -30.0, 0.0, 5.0, 8.0, -1.0])
    at = [0, 1, 31, 62, 63, 64, 69, 70, 71, 127, 128, 191, 192, 299]
    want = oracle.pooled_window_attention(q.double(), k.double(), v.double(), 1.0, torch.ones(H).double(), sink.double(), size, pool, at=at)[at]
    got = attend(kernel, q, k, v, sink, size, pool, at, bs=16, H=H, G=G, interleaved=interleaved)
    assert torch.allclose(got, want, atol=2e-5 if "f32" in kernel else 4e-2)
    assert float(want[:, 0].abs().max()) < 0.5 * float(want[:, 1].abs().max())      # the sink matters


def test_a_far_key_among_hundreds():
    """One stored average among hundreds decides the output, deep in a sequence that was decoded token by token."""
    H, G, d, dv, T, size, pool = 4, 1, 64, 64, 1500, 50, 2
    g = torch.Generator().manual_seed(2)
    q, k, v = (torch.randn(T, n, w, generator=g).bfloat16().float() * 0.1 for n, w in ((H, d), (G, d), (G, dv)))
    q[..., 0] = 4.0
    for spot in (0, 333, 777, 1440):
        kk = k.clone()
        kk[spot, 0, 0] = 16.0
        vv = v.clone()
        vv[spot] = 8.0
        want = oracle.pooled_window_attention(q.double(), kk.double(), vv.double(), 1.0, torch.ones(H).double(), torch.zeros(H).double(), size, pool, at=[T - 1])[[T - 1]]
        assert float(want.min()) > 3.5
        for kernel in ("tensor prompt", "tensor decode", "simt decode f32"):
            assert torch.allclose(attend(kernel, q, kk, vv, torch.zeros(H), size, pool, [T - 1], bs=16, H=H, G=G), want, atol=0.05)


# ------------------------------------------------------------------ whole models: prompts, portions, decoding
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompt_decode_and_portions(name, dtype):
    model, _ = model_of(name, dtype)
    t = toks(171, CONFIGS[name]["vocab"])
    want = want_logits(name, t)
    for cuts in ([], [1], [2, 4], [16, 32, 33], [23, 24, 25, 48], [169], list(range(2, 171, 2)), list(range(1, 171)),
                 [47, 48, 49, 50, 66], [7, 21, 60], [64, 128], [63, 65, 130, 131, 132, 133]):
        r = new_runner(model, graphs=len(cuts) == 170)
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
    t, want = toks(80, TENSOR["vocab"]), []
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
    lens, extra = [150, 1, 25, 70], [6, 3, 9, 1]
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
@pytest.mark.parametrize("name", list(CONFIGS))
def test_mixed_batch_of_portions_and_single_tokens(name, dtype):
    """A prompt's next portion beside decoding sequences; one waits."""
    model, _ = model_of(name, dtype)
    seqs = [toks(80, CONFIGS[name]["vocab"], seed=20 + i) for i in range(3)]
    want = [want_logits(name, s) for s in seqs]
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
    """A small pool: sequences come and go, blocks that fall behind one sequence's window serve another in the same step."""
    model, _ = model_of(name, dtype)
    vocab, lens = CONFIGS[name]["vocab"], [160, 9, 73, 150, 3, 71]
    blocks = 2 * model.init_cache(1, 1, block_size=8).blocks_for(max(lens))
    r = new_runner(model, n=2, blocks=blocks, block_size=8, graphs=True)
    live, nxt = {}, 0
    for rnd in range(16):
        while len(live) < 2:
            s = toks(lens[nxt % 6], vocab, seed=40 + nxt % 6)
            r.cache.add_sequence(nxt)
            live[nxt] = [s, 0, want_logits(name, s)]
            nxt += 1
        n = [1, 33, 2, 60][rnd % 4]
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


@pytest.mark.parametrize("dtype,name", [(F32, "odd"), (BF16, "tensor"), (F32, "tensor"), (BF16, "odd")])
def test_long_decoding(name, dtype):
    """The tables of averages outgrow their first widths, so more than one graph is captured."""
    model, _ = model_of(name, dtype)
    t = toks(400, CONFIGS[name]["vocab"], seed=9)
    r = new_runner(model, n=1, graphs=True, block_size=8)
    r.cache.add_sequence(0)
    close(feed(r, 0, t, list(range(3, 400))), want_logits(name, t), dtype)
    assert len(r.cache.tables[0]) <= r.cache.table_width and len(r._graphs) > 1


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("kind", ["recurrent", "attention"])
def test_model_of_one_kind_of_layer(kind, dtype):
    layers = {"recurrent": [mamba2(2, 24, 16, 1, 3, 2, 48), mamba2(4, 16, 10, 4, 4, 1)],
              "attention": [attention(2, 1, 24, 16, 6, 4, 24, 0.3, ff=48), attention(4, 2, 16, 10, 9, 4, 8, 0.3)]}[kind]
    cfg = config(56, 70, layers)
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
    got = LLMEngine(model, max_batch_size=2).generate([prompt, prompt], SamplingParams(max_new_tokens=4))
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
        eng = LLMEngine(model, num_blocks=60, block_size=8, max_batch_size=batch, cuda_graphs=graphs)
        assert isinstance(eng.runner, HybridRunner)
        assert eng.generate(prompts, SamplingParams(max_new_tokens=6)) == want
        assert eng.cache.pool.num_free == 60
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
    a, b = toks(80, ODD["vocab"], seed=1), toks(12, ODD["vocab"], seed=2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:78], "want": [0, 77]}, {"id": "b", "tokens": b[:11], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[78:79], "want": []}, {"id": "b", "tokens": b[11:], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[79:], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "a", "tokens": b, "want": [11]}], "end": ["a"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(tmp_path),
                        "--max-tokens", "96"], input="\n".join(map(json.dumps, steps)) + "\n", capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    assert not os.path.exists(tmp_path / "1.f32")
    wa, wb = want_logits("odd", a), want_logits("odd", b)
    for step, want in ((0, wa[[0, 77]]), (2, wa[79:]), (3, wb[11:])):
        got = np.fromfile(tmp_path / f"{step}.f32", dtype="<f4").reshape(-1, ODD["vocab"])
        close(torch.from_numpy(got), want, getattr(torch, dtype))


def test_sizes_that_no_kernel_takes_are_refused():
    cfg = config(64, 33, [mamba2(1, 8, 300, 1, 4, 1)])
    model = make_model(cfg, make_weights(cfg), F32, "cuda")
    r = new_runner(model, n=1)
    r.cache.add_sequence(0)
    with pytest.raises(RuntimeError):
        r.step([(0, [1, 2, 3], (0,))])
