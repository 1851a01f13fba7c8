"""Serving throughput of a hybrid decoder beside the closest existing models at equal size, and its kernels beside the like
kernels of those models.

``python -m sneppx_alg_b200.benchmarks.hybrid_serving [--design rilenex|tibalorn] [--sizes 1b,7b] [--part models,kernels]
[--steps 5] [--out f.json]`` (also ``python bench.py --serve-hybrid [design]``)

Sizes: the first layers of the 1B and 7B presets, random weights, bf16: six of Rilenex (four gated-write, two parallel), eight of
Tibalorn (six Mamba-2, two attention). Beside them: a Llama of the same depth, width, heads, feed-forward and vocabulary
through the paged runner, and a Mamba-2 stack of the same depth and width whose recurrent state per layer is as large as the
recurrent layer's, through the stateful runner. Prompts are synthetic token ids; a decode step runs from ``context`` tokens of
cache or state. Times are CUDA events after warm-up over the public runner calls (host preparation of every step included);
weights and activations exceed L2 many times over.

Kernel fractions: achieved / measured copy bandwidth (bytes the operation must move) or achieved / measured cuBLAS bf16
throughput, whichever bound is nearer. Attention counts the products of visible pairs; with a folded head mix (query width
kv_heads * dim) those that every exact tensor-core form of it has to do, and ``useful`` the unmixed products only.
"""
from __future__ import annotations

import argparse
import copy
import json

import torch

from .kernels import _peaks, _time

CASES = [("prefill", 1, 4096), ("prefill", 8, 2048), ("decode", 1, 2000), ("decode", 64, 2000)]


DEPTH = {"rilenex": 6, "tibalorn": 8}


def _hybrid(design, size):
    from ..models import build_model, config_from_name
    cfg = config_from_name(f"{design}-{size}")
    n = DEPTH[design]
    cfg.layer_specs = copy.deepcopy(cfg.layer_specs[:n])
    cfg.num_hidden_layers = cfg.num_layers = n
    return build_model(cfg, dtype=torch.bfloat16, device="cuda"), cfg


def _llama(cfg):
    from ..models import ModelConfig, build_model
    m = next(s for s in cfg.layer_specs if s["type"] in ("parallel", "attention"))
    a = m["mixer"].get("left", m["mixer"])
    c = ModelConfig(architecture="transformer", hidden_size=cfg.hidden_size, num_hidden_layers=cfg.num_hidden_layers,
                    num_attention_heads=a["heads"], num_key_value_heads=a["kv_heads"], head_dim=a["dim"], intermediate_size=m["mlp"]["ff"],
                    vocab_size=cfg.vocab_size, max_position_embeddings=8192)
    return build_model(c, dtype=torch.bfloat16, device="cuda").eval(), c


def _mamba(cfg):
    from ..models import ModelConfig, build_model
    m = cfg.layer_specs[0]["mixer"]
    expand, groups = (1, 8) if cfg.architecture == "rilenex" else (m["heads"] * m["vdim"] // cfg.hidden_size, m["groups"])
    c = ModelConfig(architecture="mamba2", hidden_size=cfg.hidden_size, num_hidden_layers=cfg.num_hidden_layers, vocab_size=cfg.vocab_size,
                    ssm_state_size=128, ssm_expand=expand, ssm_head_dim=64, ssm_ngroups=groups, ssm_conv_kernel=4, max_position_embeddings=8192)
    return build_model(c, dtype=torch.bfloat16, device="cuda").eval(), c


def _time_model(kind, model, cfg, case, B, T, steps):
    from ..serving.hybrid_runner import HybridRunner
    from ..serving.kv_cache import PagedKVCache
    from ..serving.llm_engine import LlamaPagedRunner, StatefulRunner
    prompts = [[(7 * i + b) % cfg.vocab_size for i in range(T)] for b in range(B)]
    ids = list(range(B))
    if kind == "mamba2":
        r = StatefulRunner(model)
        if case == "prefill":
            def fn():
                for b in ids:
                    r.prefill(b, prompts[b], 0)
        else:
            r.prefill(0, prompts[0], 0)
            for b in ids[1:]:
                r.states[b] = r.states[0]

            def fn():
                r.decode(ids, [5] * B)
    else:
        if hasattr(model, "init_cache"):
            r = HybridRunner(model, model.init_cache(B, max_tokens=T + 4 * steps + 48))
        else:
            blocks = B * ((T + 4 * steps + 63) // 16 + 1)
            r = LlamaPagedRunner(model, PagedKVCache(cfg.num_hidden_layers, blocks, 16, cfg.num_key_value_heads, cfg.head_dim, device="cuda", enable_prefix_cache=False))
        if case == "prefill":
            def fn():
                for b in ids:
                    r.cache.add_sequence(b)
                r.prefill_batch(ids, prompts) if B > 1 else r.prefill(0, prompts[0], 0)
                for b in ids:
                    r.cache.free_sequence(b)
        else:
            for b in ids:
                r.cache.add_sequence(b)
                r.cache.reserve(b, T)      # cache contents do not matter for the time
            r.enable_graphs(B, T + 4 * steps + 48)

            def fn():
                r.decode(ids, [5] * B)
    with torch.no_grad():
        ms = _time(fn, steps if case == "prefill" else 2 * steps)
    from ..ops import check_status
    check_status()
    return ms, B * (T if case == "prefill" else 1) / ms * 1e3


def bench_models(design, sizes, steps):
    out = []
    for size in sizes:
        ours, cfg = _hybrid(design, size)
        for kind in (design, "llama", "mamba2"):
            model, c = (ours, cfg) if kind == design else (_llama(cfg) if kind == "llama" else _mamba(cfg))
            n = sum(p.numel() for p in model.parameters())
            for case, B, T in CASES:
                ms, tps = _time_model(kind, model, c, case, B, T, steps)
                out.append(dict(size=size, model=kind, parameters=n, case=case, batch=B, tokens=T, ms=round(ms, 4), tokens_per_s=round(tps)))
                print(json.dumps(out[-1]), flush=True)
            del model
            torch.cuda.empty_cache()
        del ours
    return out


# ----------------------------------------------------------------------------- kernels
class _Table:
    """Collects kernel measurements and prints each as a JSON line."""

    def __init__(self):
        self.hbm, self.tf, self.src = _peaks()
        self.rows = []

    def __call__(self, name, ms, nbytes, flops=0.0, **kw):
        frac = max(nbytes / ms / 1e6 / self.hbm, flops / ms / 1e9 / self.tf)
        self.rows.append(dict(kernel=name, ms=round(ms, 4), bytes=int(nbytes), flops=int(flops), **{f"frac_of_{self.src}": round(frac, 3)}, **kw))
        print(json.dumps(self.rows[-1]), flush=True)


def _decode_batch(cache, n, ctx):
    """Decode batch of ``n`` sequences at ``ctx`` tokens each."""
    from ..ops.ragged import RaggedBatch
    for i in range(n):
        cache.add_sequence(i)
        cache.reserve(i, ctx)
    pos = [cache.lens[i] for i in range(n)]
    ent = [cache.reserve(i, 1)[0] for i in range(n)]
    width = cache.table_width
    pw = max((len(t[0]) for t in cache.averages.values()), default=0)
    pools = {p: ([-1] * n, [cache.averages[p][i] for i in range(n)]) for p in cache.pools}
    host = torch.zeros(RaggedBatch.decode_layout(n, width, cache.pools, pw)[1], dtype=torch.int32)
    RaggedBatch.fill_decode(host.numpy(), n, width, [5] * n, pos, [cache.slots[i] for i in range(n)], ent, [cache.tables[i] for i in range(n)],
                            [cache.base[i] for i in range(n)], pools, pw)
    return RaggedBatch.decode_views(host.cuda(), n, width, cache.pools, pw)


def bench_tibalorn_kernels(steps, B=8, T=4096, NB=64, ctx=8000):
    """1B sizes: prompt kernels on B x T rows, decode kernels on NB sequences at ``ctx`` tokens."""
    from ..ops import functional as F
    from ..ops import hybrid, paged, ssm
    from ..ops.ragged import RaggedBatch
    model, cfg = _hybrid("tibalorn", "1b")
    add, bf, it = _Table(), dict(dtype=torch.bfloat16, device="cuda"), 4 * steps
    rows, w = B * T, cfg.hidden_size
    mam, att = model.layers[0].mixer, model.layers[3].mixer
    s, a = mam.branches[0], att.branches[0]
    H, P, N, G, taps = s.H, s.P, s.N, s.G, s.taps
    win = a.window
    cache = model.init_cache(NB, max_tokens=ctx + 64)
    b = RaggedBatch.prompt("cuda", [[1] * T] * B, [0] * B, list(range(B)), [[-1] * T] * B, {win: [[]] * B}, [0],
                           averages={win: [([], list(range(T // win.pool)))] * B})
    with torch.no_grad():
        x = torch.randn(rows, w, device="cuda")
        n1 = model.layers[0].norm1
        add("layer norm, fp32 residual in", _time(lambda: n1(x, torch.bfloat16), it), rows * w * 6)
        xb, wb = torch.randn(rows, w, **bf), torch.ones(w, **bf)
        add("like: rmsnorm + residual (bf16)", _time(lambda: F.rmsnorm(xb, wb, 1e-5, residual=xb), it), rows * w * 8)
        del x, xb

        # recurrence over prompts
        u, y = torch.randn(rows, mam.in_proj.shape[0], **bf), torch.empty(rows, H * P, **bf)
        st = cache.state[0]
        args = (u, s.conv, s.conv_bias, st["ring"], s.dt_bias, s.a_log, s.skip, st["S"], y, b, H, P, N, G, taps)
        ops = hybrid.ssd_operands(*args)
        add("ssd operands (conv, step sizes)", _time(lambda: hybrid.ssd_operands(*args), it), rows * (s.channels * 4 + H * 10))
        xc, wc = torch.randn(B, T, s.channels, **bf), torch.randn(s.channels, 4, **bf)
        add("like: causal conv1d + silu", _time(lambda: ssm.causal_conv1d(xc, wc), it), rows * s.channels * 4)
        del xc
        add("ssd scan (gate and skip included)", _time(lambda: hybrid.ssd_scan(ops, b), it), rows * (3 * H * P + 2 * G * N + 4 * H) * 2 + B * H * N * P * 4)
        sa = (torch.randn(B, T, H, P, **bf), torch.rand(B, T, H, device="cuda") * 0.1, -torch.rand(H, device="cuda"), torch.randn(B, T, G, N, **bf),
              torch.randn(B, T, G, N, **bf), torch.ones(H, device="cuda"))
        add("like: SSD scan (Mamba-2)", _time(lambda: ssm.ssd_scan(*sa, chunk=128), it), rows * (2 * H * P + 2 * G * N + 2 * H) * 2 + B * H * N * P * 4)
        del sa
        add("norm of parts, in place", _time(lambda: hybrid.part_rmsnorm_(y, s.norm, s.parts, 1e-5), it), rows * H * P * 4)
        yb, wb = torch.randn(rows, H * P, **bf), torch.ones(H * P, **bf)
        add("like: rmsnorm (bf16)", _time(lambda: F.rmsnorm(yb, wb, 1e-5), it), rows * H * P * 4)
        del u, y, ops, args, yb

        # attention over prompts
        H, G, d, dv = a.H, a.G, a.d, a.dv
        view, c = b.views[win], (H + G) * d + G * dv
        up, yo = torch.randn(rows, att.in_proj.shape[0], **bf), torch.empty(rows, H * dv, **bf)
        qkv, gate = up[:, :c], up[:, att.where[0]["g"]: att.where[0]["g"] + H * dv]
        q, k, v = torch.empty(rows, H, d, **bf), torch.zeros(view.rows, G * d, **bf), torch.zeros(view.rows, G * dv, **bf)
        pre = lambda: hybrid.win_prep(qkv, a.bias, *a.freqs(up.device), a.rot_mul, a.temp, b, cache.k[0], cache.v[0], H, G, d, dv, q=q, k_out=k,  # noqa: E731
                                      v_out=v, dp=d, dvp=dv, kv_row=view.kv_row)
        turn = pre()
        add("attention operands (bias, rotations, angle table)", _time(pre, it), rows * (4 * c + dv * 4))
        cos, sin = F.rope_tables(T, d, 5e5, "cuda")
        qkv4 = torch.randn(B, T, c, **bf)
        add("like: RoPE (out of place)", _time(lambda: F.rope_qk_(qkv4, cos, sin, H + G, d), it), rows * ((H + G) * d + c) * 4)
        add("block averages (keys)", _time(lambda: hybrid.pool_blocks(k, d, cache.k[0], view, G, d, win.pool), it), rows * G * d * 2 * (1 + 2 / win.pool))
        full = sum(min(i + 1, win.size) + win.blocks_seen(i) for i in range(T)) * B * H
        add("window attention, prompt", _time(lambda: hybrid.window_attention(k, v, d, dv, a.sink, turn, gate, yo, b, view, a.scale, H, G, d, dv, win, q=q), it),
            0, full * 2 * (d + dv))
        q4, k4, v4 = torch.randn(B, T, H, d, **bf), torch.randn(B, T, G, d, **bf), torch.randn(B, T, G, dv, **bf)
        band = sum(min(i + 1, win.size) for i in range(T)) * B * H
        add("like: flash attention with the same window", _time(lambda: F.attention(q4, k4, v4, causal=True, window=win.size), it), 0, band * 2 * (d + dv))
        add("like: flash attention, causal", _time(lambda: F.attention(q4, k4, v4, causal=True), it), 0, B * T * (T + 1) / 2 * H * 2 * (d + dv))
        del q4, k4, v4, qkv4, up, q, k, v, yo

        # decode
        db = _decode_batch(cache, NB, ctx)
        u1 = torch.randn(NB, mam.in_proj.shape[0], **bf)
        yd = torch.empty(NB, s.out_width, **bf)
        add("ssd decode step (state of all sequences)", _time(lambda: hybrid.ssd_step(u1, s.conv, s.conv_bias, st["ring"], s.dt_bias, s.a_log, s.skip, st["S"], yd,
                                                                                     db, s.H, P, N, s.G, taps), it), NB * s.H * N * P * 8)
        u2 = torch.randn(NB, att.in_proj.shape[0], **bf)
        qkv, gate, q = u2[:, :c], u2[:, att.where[0]["g"]: att.where[0]["g"] + H * dv], torch.empty(NB, H, d, **bf)
        pre = lambda: hybrid.win_prep(qkv, a.bias, *a.freqs(u2.device), a.rot_mul, a.temp, db, cache.k[0], cache.v[0], H, G, d, dv, q=q, pool=win.pool)  # noqa: E731
        turn = pre()
        add("attention operands, decode", _time(pre, it), NB * (4 * c + dv * 4), note="launch bound")
        seen = win.size + win.blocks_seen(ctx)
        kv = NB * seen * G * (d + dv) * 2
        add("window attention, decode", _time(lambda: hybrid.window_decode(cache.k[0], cache.v[0], a.sink, turn, gate, yd[:, :H * dv], db, a.scale, H, G, d, dv, win, q=q), it), kv)
        wdt = (seen + 15) // 16
        kc, vc = torch.randn(NB * wdt, 16, G, d, **bf), torch.randn(NB * wdt, 16, G, dv, **bf)
        bt = torch.arange(NB * wdt, dtype=torch.int32, device="cuda").view(NB, wdt)
        lens = torch.full((NB,), seen, dtype=torch.int32, device="cuda")
        add("like: paged decode attention, as many keys", _time(lambda: paged.paged_decode(q, kc, vc, bt, lens), it), kv)
    return add.rows


def bench_rilenex_kernels(steps, B=8, T=2048, NB=64, ctx=2000):
    """1B sizes: prompt kernels on B x T rows, decode kernels on NB sequences at ``ctx`` tokens."""
    from ..ops import functional as F
    from ..ops import hybrid, paged, ssm
    from ..ops.ragged import RaggedBatch
    add = _Table()
    model, cfg = _hybrid("rilenex", "1b")
    rows, bf = B * T, dict(dtype=torch.bfloat16, device="cuda")
    w, it = cfg.hidden_size, 4 * steps
    gate, par = model.layers[0].mixer, model.layers[2].mixer
    g, (at, de) = gate.branches[0], par.branches
    H, d, dv, G = at.H, at.d, at.dv, at.G
    cache = model.init_cache(NB)
    b = RaggedBatch.prompt("cuda", [[1] * T] * B, [0] * B, list(range(B)), [[-1] * T] * B, {at.chunk: [[]] * B}, [0])
    x = torch.randn(rows, w, device="cuda")
    ug, up = torch.randn(rows, gate.in_proj.shape[0], **bf), torch.randn(rows, par.in_proj.shape[0], **bf)
    y = torch.empty(rows, par.out_proj.shape[1], **bf)
    with torch.no_grad():
        add("rmsnorm, fp32 residual in", _time(lambda: hybrid.rmsnorm_f32(x, model.norm.weight, 1e-5, torch.bfloat16), it), rows * w * 6)
        xb, wb = torch.randn(rows, w, **bf), torch.ones(w, **bf)
        add("like: rmsnorm + residual (bf16)", _time(lambda: F.rmsnorm(xb, wb, 1e-5, residual=xb), it), rows * w * 8)

        # recurrences: the projections in, the read-outs out; the state is read and written once
        q, f, v = (ug[:, gate.where[0][n]: gate.where[0][n] + g.segments[n]] for n in ("q", "f", "v"))
        S = cache.state[0]["S"]
        io = rows * H * (2 * d + dv) * 2 + rows * H * dv * 4
        prep = lambda: hybrid.gate_chunks(q, f, g.f_bias, g.lower, b, g.H, g.d)  # noqa: E731
        rec = prep()
        rb = rec.numel() * 4
        add("gated write: chunk records", _time(prep, it), rows * H * 2 * d * 2 + rb)
        ms1 = _time(lambda: hybrid.recur_scan(rec, v, S, b, g.H, g.d, g.dv, False), it)
        add("gated write: scan", ms1, rb + rows * H * dv * 6, 3 * 2.0 * rows * H * 2 * d * dv, note="three TF32 products per fp32 product")
        add("gated write: both, ideal single pass", ms1 + _time(prep, it), io)
        del rec
        s = par.where[1]
        qkv = up[:, s["q"]: s["q"] + de.channels]
        low = torch.randn(rows, de.low2.shape[0], **bf)
        prep = lambda: hybrid.delta_chunks(qkv, de.conv, cache.state[2]["right.ring"], up[:, s["b"]: s["b"] + H], low, de.a_log, de.dt_bias, b,  # noqa: E731
                                           de.H, de.G, de.d, de.dv, de.taps)
        rec, vv = prep()
        rb = rec.numel() * 4
        add("delta rule: convolution + chunk records", _time(prep, it), rows * (de.channels + H * d + H * dv) * 2 + rb)
        ms1 = _time(lambda: hybrid.recur_scan(rec, vv, cache.state[2]["right.S"], b, de.H, de.d, de.dv, True), it)
        add("delta rule: scan", ms1, rb + rows * H * dv * 6, 3 * 2.0 * rows * H * 3 * d * dv, note="three TF32 products per fp32 product")
        add("delta rule: both, ideal single pass", ms1 + _time(prep, it), rows * (de.channels + H * d) * 2 + rows * H * dv * 4)
        o = torch.randn(rows, H, dv, device="cuda")
        add("read-out norm + gate", _time(lambda: hybrid.head_norm_gate(o, de.norm, y[:, :H * dv], 1e-5, gate=low[:, H * d:]), it), rows * H * dv * 8)
        del rec, vv, o
        L, P, N, Gs = T, 64, 128, 8
        nh = H * dv // P
        args = (torch.randn(B, L, nh, P, **bf), torch.rand(B, L, nh, device="cuda") * 0.1, -torch.rand(nh, device="cuda"), torch.randn(B, L, Gs, N, **bf),
                torch.randn(B, L, Gs, N, **bf), torch.ones(nh, device="cuda"))
        add("like: SSD scan (Mamba-2), equal state", _time(lambda: ssm.ssd_scan(*args, chunk=128), it), 2 * rows * nh * P * 2 + 2 * rows * Gs * N * 2 + rows * nh * 4)
        xc, wc = torch.randn(B, T, de.channels, **bf), torch.randn(de.channels, 4, **bf)
        add("like: causal conv1d + silu", _time(lambda: ssm.causal_conv1d(xc, wc), it), rows * de.channels * 4)
        del args, xc

        # attention over prompts
        s = par.where[0]
        qkv = up[:, s["q"]: s["q"] + at.channels]
        k, vv = torch.randn(rows, G * d, **bf), torch.randn(rows, G * dv, **bf)
        qm, view = torch.randn(rows, H, G * d, **bf), b.views[at.chunk]
        gt = up[:, s["g"]: s["g"] + H]
        pre = lambda: hybrid.qkv_prep(qkv, at.conv, cache.state[2]["left.ring"], at.q_norm, at.k_norm, at.inv_freq(x.device), b, cache.k[0], cache.v[0],  # noqa: E731
                                      H, G, d, dv, at.taps, 1e-5, qmix_out=qm, talk=at.talk, k_out=k, v_out=vv, dvp=dv, kv_row=view.kv_row)
        add("attention operands (conv, norm, rotation, head mix)", _time(pre, it), rows * (2 * at.channels + H * G * d) * 2)
        pairs = B * T * (T + 1) / 2 * H
        ms1 = _time(lambda: hybrid.talking_attention_tc(qm, k, vv, gt, y[:, :H * dv], b, view, at.scale, 1.0, H, G, d, dv, dv, at.chunk), it)
        add("attention with head mix, prompt", ms1, 0, pairs * 2 * (G * d + dv), useful=round(pairs * 2 * (d + dv) / ms1 / 1e9 / add.tf, 3))
        q4, k4, v4 = torch.randn(B, T, H, d, **bf), k.view(B, T, G, d), vv.view(B, T, G, dv)
        add("like: flash attention, prompt", _time(lambda: F.attention(q4, k4, v4, causal=True), it), 0, pairs * 2 * (d + dv))
        qkv4 = torch.randn(B, T, (H + 2 * G) * d, **bf)
        cos, sin = F.rope_tables(T, d, 5e5, "cuda")
        add("like: RoPE (out of place)", _time(lambda: F.rope_qk_(qkv4, cos, sin, H + G, d), it), rows * ((H + G) + (H + 2 * G)) * d * 4)
        del up, ug, qm, qkv4, q4, y

        # decode
        db = _decode_batch(cache, NB, ctx)
        width = cache.table_width
        u1, u2 = torch.randn(NB, gate.in_proj.shape[0], **bf), torch.randn(NB, par.in_proj.shape[0], **bf)
        yd, low = torch.empty(NB, par.out_proj.shape[1], **bf), torch.randn(NB, de.low2.shape[0], **bf)
        st = NB * H * d * dv * 8
        q, f, v = (u1[:, gate.where[0][n]: gate.where[0][n] + g.segments[n]] for n in ("q", "f", "v"))
        add("gated write: decode step (state of all sequences)",
            _time(lambda: hybrid.gated_write_step(q, f, v, g.f_bias, g.lower, S, g.norm, yd[:, :H * dv], db, H, d, dv, 1e-5), it), st)
        s = par.where[1]
        add("delta rule: decode step (state of all sequences)",
            _time(lambda: hybrid.delta_step(u2[:, s["q"]: s["q"] + de.channels], de.conv, cache.state[2]["right.ring"], u2[:, s["b"]: s["b"] + H], low, de.a_log,
                                            de.dt_bias, cache.state[2]["right.S"], de.norm, yd[:, :H * dv], db, H, de.G, d, dv, de.taps, 1e-5,
                                            gate=low[:, H * d:]), it), st)
        qm = torch.randn(NB, H, G * d, **bf)
        gt = u2[:, par.where[0]["g"]: par.where[0]["g"] + H]
        kv = NB * (ctx % at.chunk + 1) * G * (d + dv) * 2
        add("attention with head mix, decode",
            _time(lambda: hybrid.talking_decode(None, cache.k[0], cache.v[0], at.talk, gt, yd[:, :H * dv], db, at.scale, 1.0, H, G, d, dv, at.chunk, qmix=qm), it), kv)
        bt = db.block_table.view(NB, width)
        lens = torch.full((NB,), ctx + 1, dtype=torch.int32, device="cuda")
        qd = torch.randn(NB, H, d, **bf)
        add("like: paged decode attention", _time(lambda: paged.paged_decode(qd, cache.k[0], cache.v[0], bt, lens), it), kv)
    return add.rows


def main(argv=None):
    ap = argparse.ArgumentParser(description=__doc__.split("\n")[0])
    ap.add_argument("--design", default="rilenex", choices=sorted(DEPTH))
    ap.add_argument("--sizes", default="1b,7b")
    ap.add_argument("--part", default="models,kernels")
    ap.add_argument("--steps", type=int, default=5)
    ap.add_argument("--out")
    a = ap.parse_args(argv)
    parts = a.part.split(",")
    out = {}
    if "kernels" in parts:
        out["kernels"] = (bench_rilenex_kernels if a.design == "rilenex" else bench_tibalorn_kernels)(a.steps)
        torch.cuda.empty_cache()
    if "models" in parts:
        out["models"] = bench_models(a.design, a.sizes.split(","), a.steps)
    if a.out:
        with open(a.out, "w") as f:
            json.dump(out, f, indent=1)
    return out


if __name__ == "__main__":
    main()
