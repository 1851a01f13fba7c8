"""Front-ends of the hybrid-decoder kernels: fp32-residual norms, the gated recurrences (``csrc/recurrence.cu``), the SSD
recurrence (``csrc/ssd_serve.cu``), chunked attention with a head mix before the softmax (``csrc/talking_attn.cu``), and window
attention over tokens and averaged blocks (``csrc/window_attn.cu``). They run on CUDA tensors only; activations are bf16 or
fp32, everything that the recurrences and the softmax work on is fp32 inside."""
from __future__ import annotations

import ctypes as C

import torch

from . import _lib
from ._lib import c_float, c_int, c_ll, ptr, stream
from .ragged import RaggedBatch


def _f32(t) -> int:
    if t.dtype == torch.float32:
        return 1
    if t.dtype == torch.bfloat16:
        return 0
    raise TypeError(f"activation type {t.dtype} is not supported (bfloat16 or float32)")


def _need_cuda(t):
    if not t.is_cuda:
        raise RuntimeError("this operation runs on a CUDA device only")
    _lib.lib()


def embed_f32(table, ids, scale=1.0):
    """fp32 rows of the embedding table, times ``scale``."""
    _need_cuda(table)
    x = torch.empty(ids.numel(), table.shape[1], dtype=torch.float32, device=table.device)
    _lib.call("sx_embed_f32", ptr(table), ptr(ids), ptr(x), c_int(ids.numel()), c_int(table.shape[1]), c_float(scale),
              c_int(_f32(table)), stream())
    return x


def rmsnorm_f32(x, w, eps, out_dtype, rows=None):
    """RMSNorm of fp32 rows (all of them, or the listed ones) into activations."""
    _need_cuda(x)
    n = x.shape[0] if rows is None else rows.numel()
    y = torch.empty(n, x.shape[1], dtype=out_dtype, device=x.device)
    _lib.call("sx_rmsnorm_f32", ptr(x), ptr(w), ptr(rows), ptr(y), c_int(n), c_int(x.shape[1]), c_float(eps), c_int(_f32(y)), stream())
    return y


def layernorm_f32(x, w, b, eps, out_dtype, rows=None):
    """Layer norm with weight and bias of fp32 rows (all of them, or the listed ones) into activations."""
    _need_cuda(x)
    n = x.shape[0] if rows is None else rows.numel()
    y = torch.empty(n, x.shape[1], dtype=out_dtype, device=x.device)
    _lib.call("sx_layernorm_f32", ptr(x), ptr(w), ptr(b), ptr(rows), ptr(y), c_int(n), c_int(x.shape[1]), c_float(eps), c_int(_f32(y)),
              stream())
    return y


def part_rmsnorm_(y, w, parts, eps):
    """RMS norm of ``parts`` equal parts of every row of y (a column slice will do), in place."""
    _lib.call("sx_part_rmsnorm", ptr(y), c_ll(y.stride(0)), ptr(w), c_int(y.shape[0]), c_int(y.shape[1]), c_int(parts), c_float(eps),
              c_int(_f32(y)), stream())


def head_norm_gate(o, w, y, eps, gate=None, mul=1.0):
    """y[t, h] = o[t, h] / rms * w * sigmoid(gate) * mul per head; o [T, H, dv] fp32, y [T, H * dv] (a column slice will do)."""
    T, H, dv = o.shape
    _lib.call("sx_head_norm_gate", ptr(o), ptr(w), ptr(gate), c_ll(gate.stride(0) if gate is not None else 0), c_float(mul),
              ptr(y), c_ll(y.stride(0)), c_int(T), c_int(H), c_int(dv), c_float(eps), c_int(_f32(y)), stream())


def conv_ring(u, ring, batch: RaggedBatch, channels, taps):
    """Keep the last ``taps - 1`` projected rows of every portion in its slot's ring."""
    if taps > 1:
        r = batch.struct()
        _lib.call("sx_conv_ring", ptr(u), c_ll(u.stride(0)), ptr(ring), C.byref(r), c_int(channels), c_int(taps), c_int(_f32(u)), stream())


# ----------------------------------------------------------------------------- recurrences
def _records(batch, H, d, delta, device):
    n = _lib.lib().sx_recur_record(c_int(d), c_int(int(delta)))
    return torch.empty(batch.n_chunks * H * n, dtype=torch.float32, device=device)


def gate_chunks(qr, fr, bias, lower, batch: RaggedBatch, H, d):
    """State-independent operands of a gated-write recurrence (q = silu, lower-bounded forget gate) for ``recur_scan``."""
    _need_cuda(qr)
    assert qr.stride(0) == fr.stride(0)
    rec = _records(batch, H, d, False, qr.device)
    a = _lib.SxGateArgs()
    a.q, a.f, a.ld, a.bias, a.lower, a.rec = qr.data_ptr(), fr.data_ptr(), qr.stride(0), bias.data_ptr(), lower.data_ptr(), rec.data_ptr()
    a.ragged, a.chunks, a.H, a.d, a.f32 = batch.struct(), batch.chunks(), H, d, _f32(qr)
    _lib.call("sx_gate_chunks", C.byref(a), stream())
    return rec


def _delta_args(u, wconv, ring, b, a, a_log, dt_bias, batch, H, G, d, dv, taps):
    x = _lib.SxDeltaArgs()
    x.u, x.u_ld, x.wconv, x.ring = u.data_ptr(), u.stride(0), wconv.data_ptr(), ring.data_ptr()
    x.b, x.b_ld, x.a, x.a_ld = b.data_ptr(), b.stride(0), a.data_ptr(), a.stride(0)
    x.a_log, x.dt_bias = a_log.data_ptr(), dt_bias.data_ptr()
    x.ragged = batch.struct()
    x.T, x.H, x.G, x.d, x.dv, x.taps, x.f32 = batch.T, H, G, d, dv, taps, _f32(u)
    return x


def delta_chunks(u, wconv, ring, b, a, a_log, dt_bias, batch: RaggedBatch, H, G, d, dv, taps):
    """State-independent operands of the gated delta rule for ``recur_scan``, and the convolved values [T, H * dv]."""
    _need_cuda(u)
    rec = _records(batch, H, d, True, u.device)
    v = torch.empty(batch.T, H * dv, dtype=u.dtype, device=u.device)
    x = _delta_args(u, wconv, ring, b, a, a_log, dt_bias, batch, H, G, d, dv, taps)
    x.v = v.data_ptr()
    ch = batch.chunks()
    _lib.call("sx_delta_chunks", C.byref(x), C.byref(ch), ptr(rec), stream())
    return rec, v


def recur_scan(rec, v, state, batch: RaggedBatch, H, d, dv, delta):
    """Walks every portion of the batch from its slot's state (empty at position 0), stores the state back and returns the
    read-outs [T, H, dv] fp32."""
    o = torch.empty(batch.T, H, dv, dtype=torch.float32, device=v.device)
    x = _lib.SxScanArgs()
    x.rec, x.v, x.v_ld, x.state, x.o = rec.data_ptr(), v.data_ptr(), v.stride(0), state.data_ptr(), o.data_ptr()
    x.ragged, x.chunks, x.status = batch.struct(), batch.chunks(), _lib.status_word(v.device).data_ptr()
    x.H, x.d, x.dv, x.delta, x.f32 = H, d, dv, int(delta), _f32(v)
    _lib.call("sx_recur_scan", C.byref(x), stream())
    return o


def _step_args(state, norm, y, batch, H, Hq, d, dv, eps, gate, mul):
    s = _lib.SxStepArgs()
    s.state, s.norm, s.y, s.y_ld = state.data_ptr(), norm.data_ptr(), y.data_ptr(), y.stride(0)
    if gate is not None:
        s.gate, s.gate_ld = gate.data_ptr(), gate.stride(0)
    s.ragged = batch.struct()
    s.mul, s.eps = mul, eps
    s.H, s.Hq, s.d, s.dv, s.f32 = H, Hq, d, dv, _f32(y)
    return s


def gated_write_step(qr, fr, vr, bias, lower, state, norm, y, batch: RaggedBatch, H, d, dv, eps, gate=None, mul=1.0):
    """One token of every sequence through the gated-write recurrence, from projected rows to normed read-outs in y."""
    _need_cuda(qr)
    s = _step_args(state, norm, y, batch, H, H, d, dv, eps, gate, mul)
    s.qr, s.fr, s.vr, s.ld = qr.data_ptr(), fr.data_ptr(), vr.data_ptr(), qr.stride(0)
    s.fbias, s.lower, s.delta = bias.data_ptr(), lower.data_ptr(), 0
    _lib.call("sx_recur_step", C.byref(s), stream())


def delta_step(u, wconv, ring, b, a, a_log, dt_bias, state, norm, y, batch: RaggedBatch, H, G, d, dv, taps, eps, gate=None, mul=1.0):
    """One token of every sequence through the gated delta rule, from projected rows to gated read-outs in y."""
    _need_cuda(u)
    s = _step_args(state, norm, y, batch, H, G, d, dv, eps, gate, mul)
    s.inp = _delta_args(u, wconv, ring, b, a, a_log, dt_bias, batch, H, G, d, dv, taps)
    s.delta = 1
    _lib.call("sx_recur_step", C.byref(s), stream())


# ----------------------------------------------------------------------------- SSD recurrence
def _ssd_args(u, wconv, bconv, ring, dt_bias, a_log, D, state, y, batch, H, P, N, G, taps):
    a = _lib.SxSsdArgs()
    a.u, a.u_ld, a.wconv, a.bconv, a.ring = u.data_ptr(), u.stride(0), wconv.data_ptr(), bconv.data_ptr(), ring.data_ptr()
    a.dt_bias, a.a_log, a.D, a.state, a.y, a.y_ld = (dt_bias.data_ptr(), a_log.data_ptr(), D.data_ptr(), state.data_ptr(), y.data_ptr(),
                                                     y.stride(0))
    a.ragged = batch.struct()
    if not batch.decode:
        a.chunks = batch.chunks()
    a.T, a.H, a.P, a.N, a.G, a.taps, a.xp, a.np, a.f32 = batch.T, H, P, N, G, taps, P, N, _f32(u)
    return a


def ssd_scan_tc(act_dtype, P, N) -> bool:
    """Whether the tensor-core prompt kernel takes these sizes."""
    return act_dtype == torch.bfloat16 and bool(_lib.lib().sx_ssd_scan_ok(c_int(P), c_int(N)))


def ssd_operands(u, wconv, bconv, ring, dt_bias, a_log, D, state, y, batch: RaggedBatch, H, P, N, G, taps):
    """Convolved x, B, C, step sizes and decays of the rows of a prompt batch, from projected rows (z | x | B | C | dt). Returns
    what ``ssd_scan`` takes: the kernels' arguments and the tensors that they point to."""
    _need_cuda(u)
    T, dev = batch.T, u.device
    a = _ssd_args(u, wconv, bconv, ring, dt_bias, a_log, D, state, y, batch, H, P, N, G, taps)
    if ssd_scan_tc(u.dtype, P, N):
        a.xp, a.np = (P + 7) // 8 * 8, (N + 7) // 8 * 8
    x = torch.empty(T, H * a.xp, dtype=u.dtype, device=dev)
    b, c = torch.empty(2, T, (G * a.np + 7) // 8 * 8, dtype=u.dtype, device=dev)
    dt, la = torch.empty(2, T, H, dtype=torch.float32, device=dev)
    a.x, a.b, a.c, a.dt, a.la = x.data_ptr(), b.data_ptr(), c.data_ptr(), dt.data_ptr(), la.data_ptr()
    _lib.call("sx_ssd_operands", C.byref(a), stream())
    return a, (u, x, b, c, dt, la, state, y, D)


def ssd_scan(operands, batch: RaggedBatch):
    """Walks every portion of the batch from its slot's state (empty at position 0), stores the state back and writes the gated
    read-outs."""
    a, (u, x, _, _, _, _, state, _, _) = operands
    if ssd_scan_tc(u.dtype, a.P, a.N):
        # segments cost a pass over the states: worth it while one CTA per portion and head leaves a third of the SMs idle
        if batch.n_segments > batch.n and batch.n * a.H * ((a.P + 63) // 64) <= 100:
            seg = torch.empty(batch.n_segments * a.H * (a.N * a.P + 1), dtype=torch.float32, device=u.device)
            a.seg_seq, a.seg_first, a.seg_state = batch.seg_seq.data_ptr(), batch.seg_first.data_ptr(), seg.data_ptr()
            a.seg_la = seg.data_ptr() + 4 * batch.n_segments * a.H * a.N * a.P
            a.n_seg, a.seg_rows = batch.n_segments, batch.segment_rows
        _lib.call("sx_ssd_scan", C.byref(a), stream())
        return
    rec = _records(batch, a.H, a.N, False, u.device)
    _lib.call("sx_ssd_chunks", C.byref(a), ptr(rec), stream())
    o = recur_scan(rec, x, state, batch, a.H, a.N, a.P, delta=False)
    _lib.call("sx_ssd_gate", C.byref(a), ptr(o), stream())


def ssd_prompt(u, wconv, bconv, ring, dt_bias, a_log, D, state, y, batch: RaggedBatch, H, P, N, G, taps):
    """Portions through the SSD recurrence, from projected rows to gated read-outs in y."""
    operands = ssd_operands(u, wconv, bconv, ring, dt_bias, a_log, D, state, y, batch, H, P, N, G, taps)
    conv_ring(u[:, H * P:], ring, batch, H * P + 2 * G * N, taps)
    ssd_scan(operands, batch)


def ssd_step(u, wconv, bconv, ring, dt_bias, a_log, D, state, y, batch: RaggedBatch, H, P, N, G, taps):
    """One token of every sequence through the SSD recurrence, from projected rows to gated read-outs in y."""
    _need_cuda(u)
    a = _ssd_args(u, wconv, bconv, ring, dt_bias, a_log, D, state, y, batch, H, P, N, G, taps)
    _lib.call("sx_ssd_step", C.byref(a), stream())


# ----------------------------------------------------------------------------- attention with a head mix
def qkv_prep(u, wconv, ring, qn, kn, inv_freq, batch: RaggedBatch, k_cache, v_cache, H, G, d, dv, taps, eps, q_out=None,
             qmix_out=None, talk=None, k_out=None, v_out=None, dvp=0, kv_row=None):
    """Convolution, query / key norm, rotation and cache append of attention operands (see ``SxQkvArgs``)."""
    _need_cuda(u)
    x = _lib.SxQkvArgs()
    x.u, x.u_ld, x.wconv, x.ring = u.data_ptr(), u.stride(0), wconv.data_ptr(), ring.data_ptr()
    x.qn, x.kn, x.inv_freq = qn.data_ptr(), kn.data_ptr(), inv_freq.data_ptr()
    for name, t in (("talk", talk), ("q_out", q_out), ("qmix_out", qmix_out), ("k_out", k_out), ("v_out", v_out), ("kv_row", kv_row)):
        if t is not None:
            setattr(x, name, t.data_ptr())
    if qmix_out is not None:
        x.qmix_ld = qmix_out.shape[-1]
    if k_out is not None:
        x.k_ld, x.v_ld = k_out.stride(0), v_out.stride(0)
    x.k_cache, x.v_cache, x.cache_entry = k_cache.data_ptr(), v_cache.data_ptr(), batch.entry.data_ptr()
    x.ragged = batch.struct()
    x.T, x.H, x.G, x.d, x.dv, x.dvp, x.taps = batch.T, H, G, d, dv, dvp or dv, taps
    x.rot, x.f32, x.eps = 2 * inv_freq.numel(), _f32(u), eps
    if not batch.decode:
        x.chunks = batch.chunks()
    _lib.call("sx_qkv_prep", C.byref(x), stream())


def kv_gather(cache, entry, row, out, G, w, wp):
    """Copy cache entries (earlier positions of the running chunk) in front of a portion's packed rows."""
    n = entry.numel()
    if n:
        _lib.call("sx_kv_gather", ptr(cache), ptr(entry), ptr(row), c_int(n), ptr(out), c_ll(out.stride(0)), c_int(G), c_int(w),
                  c_int(wp), c_int(_f32(cache)), stream())


def _talk_args(q, k, v, k_ld, v_ld, talk, gate, y, batch, scale, mul, H, G, d, dv, dvp, size):
    a = _lib.SxTalkArgs()
    a.q, a.k, a.v, a.k_ld, a.v_ld, a.dvp = q.data_ptr(), k.data_ptr(), v.data_ptr(), k_ld, v_ld, dvp
    a.talk, a.gate, a.gate_ld, a.y, a.y_ld = talk.data_ptr(), gate.data_ptr(), gate.stride(0), y.data_ptr(), y.stride(0)
    a.ragged = batch.struct()
    a.scale, a.mul = scale, mul
    a.T, a.H, a.G, a.d, a.dv, a.size, a.f32, a.splits = batch.T, H, G, d, dv, size, _f32(y), 1
    return a


def talking_attention(q, k, v, talk, gate, y, batch: RaggedBatch, kv_base, scale, mul, H, G, d, dv, dvp, size):
    """Prompt form over packed keys and values; q fp32 [T, H, d]; y[t, h] = o * sigmoid(gate[t, h]) * mul."""
    a = _talk_args(q, k, v, k.stride(0), v.stride(0), talk, gate, y, batch, scale, mul, H, G, d, dv, dvp, size)
    a.kv_base = kv_base.data_ptr()
    _lib.call("sx_talk_attn", C.byref(a), stream())


def talking_tc(act_dtype, H, G, d, dv) -> bool:
    """Whether the tensor-core prompt kernel takes these sizes."""
    return act_dtype == torch.bfloat16 and bool(_lib.lib().sx_talk_attn_tc_ok(c_int(H), c_int(G), c_int(d), c_int(dv)))


def talking_attention_tc(qmix, k, v, gate, y, batch: RaggedBatch, view, scale, mul, H, G, d, dv, dvp, size):
    """Tensor-core prompt form: ``qmix`` [T, H, ceil(G d / 64) * 64] from ``qkv_prep``."""
    a = _lib.SxTalkTcArgs()
    a.qmix, a.k, a.v = qmix.data_ptr(), k.data_ptr(), v.data_ptr()
    a.k_ld, a.v_ld, a.kv_rows = k.stride(0), v.stride(0), k.shape[0]
    a.kv_base, a.tiles, a.n_tiles = view.kv_base.data_ptr(), view.tiles.data_ptr(), view.n_tiles
    a.gate, a.gate_ld, a.y, a.y_ld = gate.data_ptr(), gate.stride(0), y.data_ptr(), y.stride(0)
    a.ragged = batch.struct()
    a.scale, a.mul = scale, mul
    a.T, a.H, a.G, a.d, a.dv, a.dvp, a.size = batch.T, H, G, d, dv, dvp, size
    a.status = _lib.status_word(y.device).data_ptr()
    _lib.call("sx_talk_attn_tc", C.byref(a), stream())


def decode_splits(n: int, size: int) -> int:
    """Key slices of one decode step: one CTA per SM, at least 64 keys each."""
    return max(1, min((size + 63) // 64, 148 // max(n, 1)))


def talking_decode_tc(act_dtype, H, G, d, dv) -> bool:
    """Whether the tensor-core decode kernel takes these sizes."""
    return act_dtype == torch.bfloat16 and bool(_lib.lib().sx_talk_decode_ok(c_int(H), c_int(G), c_int(d), c_int(dv)))


def talking_decode(q, k_cache, v_cache, talk, gate, y, batch: RaggedBatch, scale, mul, H, G, d, dv, size, qmix=None):
    """Decode form: one query per sequence against the block pool. Either ``q`` (fp32 [T, H, d], any sizes) or ``qmix``
    (bf16 [T, H, q_ld] from ``qkv_prep``, the tensor-core kernel)."""
    a = _talk_args(q if q is not None else qmix, k_cache, v_cache, G * d, G * dv, talk, gate, y, batch, scale, mul, H, G, d, dv, dv, size)
    a.block_table, a.block_base = batch.block_table.data_ptr(), batch.block_base.data_ptr()
    a.table_ld, a.block_size = batch.table_width, k_cache.shape[1]
    a.splits = decode_splits(batch.n, size)
    if a.splits > 1:
        part = torch.empty(batch.n * a.splits * H * (dv + 2), dtype=torch.float32, device=y.device)
        a.part = part.data_ptr()
    if qmix is not None:
        _lib.call("sx_talk_decode", C.byref(a), ptr(qmix), c_int(qmix.shape[-1]), stream())
    else:
        _lib.call("sx_talk_attn", C.byref(a), stream())


# ----------------------------------------------------------------------------- window attention over tokens and averaged blocks
def win_prep(u, bias, freq, vfreq, rot_mul, temp, batch: RaggedBatch, k_cache, v_cache, H, G, d, dv, interleaved=False, q32=None, q=None,
             k_out=None, v_out=None, dp=0, dvp=0, kv_row=None, pool=0):
    """Bias, rotation and cache append of attention operands (see ``SxWinPrepArgs``); returns the table of value angles. In
    decoding also averages the blocks of ``pool`` positions that the tokens complete."""
    _need_cuda(u)
    turn = torch.empty(batch.T, dv // 2, 2, dtype=torch.float32, device=u.device)
    a = _lib.SxWinPrepArgs()
    a.u, a.u_ld, a.freq, a.vfreq = u.data_ptr(), u.stride(0), freq.data_ptr(), vfreq.data_ptr()
    for name, t in (("bias", bias), ("temp", temp), ("q32", q32), ("q", q), ("k_out", k_out), ("v_out", v_out), ("kv_row", kv_row)):
        if t is not None:
            setattr(a, name, t.data_ptr())
    if q is not None:
        a.q_ld = q.shape[-1]
    if k_out is not None:
        a.k_ld, a.v_ld, a.dp, a.dvp = k_out.stride(0), v_out.stride(0), dp, dvp
    a.k_cache, a.v_cache, a.cache_entry, a.turn = k_cache.data_ptr(), v_cache.data_ptr(), batch.entry.data_ptr(), turn.data_ptr()
    a.ragged = batch.struct()
    if batch.decode and pool:
        a.pool_entry, a.block_table, a.block_base = batch.pool_entry[pool].data_ptr(), batch.block_table.data_ptr(), batch.block_base.data_ptr()
        a.table_ld, a.block_size, a.pool = batch.table_width, k_cache.shape[1], pool
    a.T, a.H, a.G, a.d, a.dv, a.rot, a.interleaved, a.f32 = batch.T, H, G, d, dv, 2 * freq.numel(), int(interleaved), _f32(u)
    a.rot_mul = rot_mul
    _lib.call("sx_win_prep", C.byref(a), stream())
    return turn


def pool_blocks(rows, wp, cache, view, G, w, pool):
    """Averages of the blocks that a prompt batch completes, from its packed rows (head pitch ``wp``) to their packed rows and
    cache entries."""
    if view.n_pool:
        _lib.call("sx_pool_blocks", ptr(rows), c_ll(rows.stride(0)), c_int(wp), ptr(cache), c_int(G), c_int(w), ptr(view.pool_src),
                  ptr(view.pool_row), ptr(view.pool_entry), c_int(view.n_pool), c_int(pool), c_int(_f32(rows)), stream())


def _win_args(sink, turn, gate, y, batch, scale, H, G, d, dv, window, interleaved):
    a = _lib.SxWinAttnArgs()
    a.sink, a.turn, a.gate, a.gate_ld, a.y, a.y_ld = (sink.data_ptr(), turn.data_ptr(), gate.data_ptr(), gate.stride(0), y.data_ptr(),
                                                      y.stride(0))
    a.ragged = batch.struct()
    a.scale, a.T, a.H, a.G, a.d, a.dv, a.size, a.pool = scale, batch.T, H, G, d, dv, window.size, window.pool
    a.interleaved, a.f32, a.splits = int(interleaved), _f32(y), 1
    a.status = _lib.status_word(y.device).data_ptr()
    return a


def window_tc(act_dtype, H, G, d, dv) -> bool:
    """Whether the tensor-core prompt kernel takes these sizes."""
    return act_dtype == torch.bfloat16 and bool(_lib.lib().sx_win_attn_tc_ok(c_int(H), c_int(G), c_int(d), c_int(dv)))


def window_attention(k, v, dp, dvp, sink, turn, gate, y, batch: RaggedBatch, view, scale, H, G, d, dv, window, interleaved=False, q32=None,
                     q=None):
    """Prompt form over packed keys and values. Either ``q32`` (fp32 [T, H, d], any sizes) or ``q`` (bf16 [T, H, q_ld], the
    tensor-core kernel)."""
    a = _win_args(sink, turn, gate, y, batch, scale, H, G, d, dv, window, interleaved)
    a.k, a.v, a.k_ld, a.v_ld, a.kv_rows, a.dp, a.dvp = k.data_ptr(), v.data_ptr(), k.stride(0), v.stride(0), k.shape[0], dp, dvp
    a.kv_base, a.pool_base = view.kv_base.data_ptr(), view.pool_base.data_ptr()
    if q is not None:
        a.q, a.q_ld, a.tiles, a.n_tiles = q.data_ptr(), q.shape[-1], view.tiles.data_ptr(), view.n_tiles
        _lib.call("sx_win_attn_tc", C.byref(a), stream())
    else:
        a.q32 = q32.data_ptr()
        _lib.call("sx_win_attn", C.byref(a), stream())


def window_decode_tc(act_dtype, H, G, d, dv) -> bool:
    """Whether the tensor-core decode kernel takes these sizes."""
    return act_dtype == torch.bfloat16 and bool(_lib.lib().sx_win_decode_ok(c_int(H), c_int(G), c_int(d), c_int(dv)))


def window_decode(k_cache, v_cache, sink, turn, gate, y, batch: RaggedBatch, scale, H, G, d, dv, window, interleaved=False, q32=None, q=None):
    """Decode form: one query per sequence against the block pool; ``q32`` or ``q`` as in the prompt form."""
    a = _win_args(sink, turn, gate, y, batch, scale, H, G, d, dv, window, interleaved)
    a.k, a.v, a.k_ld, a.v_ld, a.dp, a.dvp = k_cache.data_ptr(), v_cache.data_ptr(), G * d, G * dv, d, dv
    a.block_table, a.block_base, a.table_ld, a.block_size = batch.block_table.data_ptr(), batch.block_base.data_ptr(), batch.table_width, k_cache.shape[1]
    a.pool_table, a.pool_ld = batch.pool_table[window.pool].data_ptr(), batch.pool_width
    most = window.size + batch.pool_width * a.block_size
    a.splits = max(1, min((most + 127) // 128, 2 * 148 // max(batch.n * G, 1)))
    part = torch.empty(batch.n * a.splits * H * (dv + 2), dtype=torch.float32, device=y.device)
    a.part = part.data_ptr()
    if q is not None:
        a.q, a.q_ld = q.data_ptr(), q.shape[-1]
        _lib.call("sx_win_decode", C.byref(a), stream())
    else:
        a.q32 = q32.data_ptr()
        _lib.call("sx_win_attn", C.byref(a), stream())
