"""Serving throughput of the Rilenex design beside the closest existing models at equal size, and its kernels beside the
like kernels of those models.

``python -m sneppx_alg_b200.benchmarks.hybrid_serving [--sizes 1b,4k] [--part models,kernels] [--steps 5] [--out f.json]``
(also ``python bench.py --serve-hybrid``)

Sizes: six layers (four gated-write, two parallel) of the 1B and 7B presets, random weights, bf16. Beside them: a Llama of the
same depth, width, heads, feed-forward and vocabulary through the paged runner, and a Mamba-2 stack of the same depth and
width whose recurrent state per layer is as large as the gated-write layer's, through the stateful runner. Prompts are synthetic
token ids; a decode step runs from ``context`` tokens of cache or state. Times are CUDA events after warm-up over the public
runner calls (host preparation of every step included); weights and activations exceed L2 many times over.

Kernel fractions: achieved / measured copy bandwidth (bytes the operation must move) or achieved / measured cuBLAS bf16
throughput, whichever bound is nearer. The attention counts the products of the folded head mix (query width kv_heads * dim)
that every exact tensor-core form of it has to do; ``useful`` counts the unmixed products only.
"""
from __future__ import annotations

import argparse
import copy
import json

import torch

from .kernels import _peaks, _time

CASES = [("prefill", 1, 4096), ("prefill", 8, 2048), ("decode", 1, 2000), ("decode", 64, 2000)]


def _rilenex(size):
    from ..models import build_model, config_from_name
    cfg = config_from_name("rilenex-1b" if size == "1b" else "rilenex-7b")
    cfg.layer_specs = copy.deepcopy(cfg.layer_specs[:6])
    cfg.num_hidden_layers = cfg.num_layers = 6
    return build_model(cfg, dtype=torch.bfloat16, device="cuda"), cfg


def _llama(cfg):
    from ..models import ModelConfig, build_model
    a = cfg.layer_specs[2]["mixer"]["left"]
    c = ModelConfig(architecture="transformer", hidden_size=cfg.hidden_size, num_hidden_layers=6, num_attention_heads=a["heads"],
                    num_key_value_heads=a["kv_heads"], head_dim=a["dim"], intermediate_size=cfg.layer_specs[0]["mlp"]["ff"],
                    vocab_size=cfg.vocab_size, max_position_embeddings=8192)
    return build_model(c, dtype=torch.bfloat16, device="cuda").eval(), c


def _mamba(cfg):
    from ..models import ModelConfig, build_model
    c = ModelConfig(architecture="mamba2", hidden_size=cfg.hidden_size, num_hidden_layers=6, vocab_size=cfg.vocab_size, ssm_state_size=128,
                    ssm_expand=1, ssm_head_dim=64, ssm_ngroups=8, ssm_conv_kernel=4, max_position_embeddings=8192)
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
        if kind == "rilenex":
            r = HybridRunner(model, model.init_cache(B))
        else:
            blocks = B * ((T + 4 * steps + 63) // 16 + 1)
            r = LlamaPagedRunner(model, PagedKVCache(6, blocks, 16, cfg.num_key_value_heads, cfg.head_dim, device="cuda", enable_prefix_cache=False))
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


def bench_models(sizes, steps):
    out = []
    for size in sizes:
        ours, cfg = _rilenex(size)
        for kind in ("rilenex", "llama", "mamba2"):
            model, c = (ours, cfg) if kind == "rilenex" else (_llama(cfg) if kind == "llama" else _mamba(cfg))
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
def bench_kernels(steps, B=8, T=2048, NB=64, ctx=2000):
    """1B sizes: prompt kernels on B x T rows, decode kernels on NB sequences at ``ctx`` tokens."""
    from ..ops import functional as F
    from ..ops import hybrid, paged, ssm
    from ..ops.ragged import RaggedBatch
    from ..serving.hybrid_runner import HybridRunner
    hbm, tf, src = _peaks()
    model, cfg = _rilenex("1b")
    rows, bf = B * T, dict(dtype=torch.bfloat16, device="cuda")
    w, it = cfg.hidden_size, 4 * steps
    gate, par = model.layers[0].mixer, model.layers[2].mixer
    g, (at, de) = gate.branches[0], par.branches
    H, d, dv, G = at.H, at.d, at.dv, at.G
    res = []

    def add(name, ms, nbytes, flops=0.0, **kw):
        frac = max(nbytes / ms / 1e6 / hbm, flops / ms / 1e9 / tf)
        r = dict(kernel=name, ms=round(ms, 4), bytes=int(nbytes), flops=int(flops), **{f"frac_of_{src}": round(frac, 3)}, **kw)
        res.append(r)
        print(json.dumps(r), flush=True)

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
        add("attention with head mix, prompt", ms1, 0, pairs * 2 * (G * d + dv), useful=round(pairs * 2 * (d + dv) / ms1 / 1e9 / tf, 3))
        q4, k4, v4 = torch.randn(B, T, H, d, **bf), k.view(B, T, G, d), vv.view(B, T, G, dv)
        add("like: flash attention, prompt", _time(lambda: F.attention(q4, k4, v4, causal=True), it), 0, pairs * 2 * (d + dv))
        qkv4 = torch.randn(B, T, (H + 2 * G) * d, **bf)
        cos, sin = F.rope_tables(T, d, 5e5, "cuda")
        add("like: RoPE (out of place)", _time(lambda: F.rope_qk_(qkv4, cos, sin, H + G, d), it), rows * ((H + G) + (H + 2 * G)) * d * 4)
        del up, ug, qm, qkv4, q4, y

        # decode
        r = HybridRunner(model, cache)
        for i in range(NB):
            cache.add_sequence(i)
            cache.reserve(i, ctx)
        pos = [cache.lens[i] for i in range(NB)]
        ent = [cache.reserve(i, 1)[0] for i in range(NB)]
        width = cache.table_width
        host = torch.zeros(RaggedBatch.decode_layout(NB, width)[1], dtype=torch.int32)
        RaggedBatch.fill_decode(host.numpy(), NB, width, [5] * NB, pos, [cache.slots[i] for i in range(NB)], ent, [cache.tables[i] for i in range(NB)],
                                [cache.base[i] for i in range(NB)])
        db = RaggedBatch.decode_views(host.cuda(), NB, width)
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
    del r
    return res


def main(argv=None):
    ap = argparse.ArgumentParser(description=__doc__.split("\n")[0])
    ap.add_argument("--sizes", default="1b,4k")
    ap.add_argument("--part", default="models,kernels")
    ap.add_argument("--steps", type=int, default=5)
    ap.add_argument("--out")
    a = ap.parse_args(argv)
    parts = a.part.split(",")
    out = {}
    if "kernels" in parts:
        out["kernels"] = bench_kernels(a.steps)
        torch.cuda.empty_cache()
    if "models" in parts:
        out["models"] = bench_models(a.sizes.split(","), a.steps)
    if a.out:
        with open(a.out, "w") as f:
            json.dump(out, f, indent=1)
    return out


if __name__ == "__main__":
    main()
