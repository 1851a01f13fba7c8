"""Token mixers of the hybrid decoders, built from branches that share one layer input.

A branch (``GatedWriteBranch``, ``DeltaBranch``, ``SSDBranch``, ``TalkingAttentionBranch``, ``PooledAttentionBranch``) names the projections it reads, the state it
keeps per sequence and the columns it produces; ``FusedMixer`` runs any number of branches side by side: one GEMM projects
the layer input for all of them, every branch writes its read-outs (norm, gate and branch scale applied in fp32) into its
columns of one buffer, and one GEMM multiplies those with the joined output weights and adds the result to the fp32
residual in its epilogue.

Tensor names are those of the checkpoint, relative to the mixer (``tensors()``); they are views into the fused weights.
"""
from __future__ import annotations

import math
from collections import OrderedDict
from typing import Dict, List, Tuple

import torch
import torch.nn as tnn

from ..ops import hybrid
from ..ops.gemm import gemm
from ..ops.ragged import RaggedBatch
from .modules import Module


def _up(n: int, m: int = 8) -> int:
    return (n + m - 1) // m * m


def _param(*shape, dtype=None, device=None, fill=0.0, std=None):
    t = torch.empty(*shape, dtype=dtype, device=device)
    if std is not None:
        tnn.init.normal_(t, std=std)
    else:
        t.fill_(fill)
    return tnn.Parameter(t, requires_grad=False)


class Branch(Module):
    """``segments``: projection name -> rows. ``out_width``: columns this branch writes."""

    segments: "OrderedDict[str, int]"
    out_width: int

    def kv_spec(self):
        """(kv heads, key size, value size, mask) of the cached keys, or None; a chunk length stands for its mask."""
        return None

    def state_spec(self, act_dtype) -> Dict[str, Tuple[tuple, torch.dtype]]:
        return {}

    def tensors(self) -> "List[Tuple[str, torch.Tensor]]":
        """Checkpoint tensors other than the projections, as writable views."""
        return []

    def run(self, u, y, batch: RaggedBatch, state, kv, scale: float):
        raise NotImplementedError


class GatedWriteBranch(Branch):
    """HGRN2 recurrence: the forget gate decides what is kept (f) and what is written (1 - f); ``lower`` bounds f."""

    def __init__(self, heads, dim, vdim, eps, dtype=None, device=None):
        super().__init__()
        self.H, self.d, self.dv, self.eps = heads, dim, vdim, eps
        self.segments = OrderedDict(q=heads * dim, f=heads * dim, v=heads * vdim)
        self.out_width = heads * vdim
        f32 = dict(dtype=torch.float32, device=device)
        self.f_bias = _param(heads * dim, **f32)
        self.lower = _param(heads * dim, **f32)
        self.norm = _param(vdim, fill=1.0, **f32)

    def state_spec(self, act_dtype):
        return {"S": ((self.H, self.d, self.dv), torch.float32)}

    def tensors(self):
        return [("f.b", self.f_bias), ("lower", self.lower), ("norm", self.norm)]

    def run(self, u, y, batch, state, kv, scale):
        H, d, dv = self.H, self.d, self.dv
        if batch.decode:
            hybrid.gated_write_step(u["q"], u["f"], u["v"], self.f_bias, self.lower, state["S"], self.norm, y, batch, H, d, dv,
                                    self.eps, mul=scale)
            return
        rec = hybrid.gate_chunks(u["q"], u["f"], self.f_bias, self.lower, batch, H, d)
        o = hybrid.recur_scan(rec, u["v"], state["S"], batch, H, d, dv, delta=False)
        hybrid.head_norm_gate(o, self.norm, y, self.eps, mul=scale)


class DeltaBranch(Branch):
    """Gated delta rule with one decay per key channel: short convolutions with silu on q, k, v, unit-norm q and k, decay
    and output gate from low-rank products (both second factors run as one block-diagonal GEMM)."""

    def __init__(self, heads, kv_heads, dim, vdim, taps, decay_rank, gate_rank, eps, dtype=None, device=None, init_std=0.02):
        super().__init__()
        self.H, self.G, self.d, self.dv, self.taps, self.eps = heads, kv_heads, dim, vdim, taps, eps
        self.ra, self.rg = decay_rank, gate_rank
        # q, k, v are adjacent (one convolution buffer), a1 and g1 are adjacent (one low-rank operand)
        self.segments = OrderedDict(q=kv_heads * dim, k=kv_heads * dim, v=heads * vdim, b=heads, a1=decay_rank, g1=gate_rank)
        self.tight = ("q", "k", "v")
        self.out_width = heads * vdim
        self.channels = 2 * kv_heads * dim + heads * vdim
        f32 = dict(dtype=torch.float32, device=device)
        self.conv = _param(taps, self.channels, fill=1.0 / taps, **f32)
        self.a_log = _param(heads, **f32)
        self.dt_bias = _param(heads * dim, fill=-2.0, **f32)
        self.norm = _param(vdim, fill=1.0, **f32)
        self.low2 = _param(_up(heads * dim) + _up(heads * vdim), _up(decay_rank) + _up(gate_rank), dtype=dtype, device=device)
        if init_std:
            for n, t in self.tensors():
                if n in ("a2", "g2"):
                    tnn.init.normal_(t, std=init_std)

    def state_spec(self, act_dtype):
        spec = {"S": ((self.H, self.d, self.dv), torch.float32)}
        spec["ring"] = ((self.taps, self.channels), act_dtype)
        return spec

    def tensors(self):
        Gd, Hd, Hv = self.G * self.d, self.H * self.d, self.H * self.dv
        c = self.conv.data
        return [("q.conv", c[:, :Gd].t()), ("k.conv", c[:, Gd:2 * Gd].t()), ("v.conv", c[:, 2 * Gd:].t()), ("A_log", self.a_log),
                ("norm", self.norm), ("a2", self.low2.data[:Hd, :self.ra]), ("dt_bias", self.dt_bias),
                ("g2", self.low2.data[_up(Hd): _up(Hd) + Hv, _up(self.ra): _up(self.ra) + self.rg])]

    def run(self, u, y, batch, state, kv, scale):
        H, G, d, dv = self.H, self.G, self.d, self.dv
        low = gemm(u.span("a1", "g1", _up(self.ra) + _up(self.rg)), self.low2)
        a, gate = low[:, :H * d], low[:, _up(H * d): _up(H * d) + H * dv]
        qkv = u["q"]
        if batch.decode:
            hybrid.delta_step(qkv, self.conv, state["ring"], u["b"], a, self.a_log, self.dt_bias, state["S"], self.norm, y, batch,
                              H, G, d, dv, self.taps, self.eps, gate=gate, mul=scale)
            return
        rec, v = hybrid.delta_chunks(qkv, self.conv, state["ring"], u["b"], a, self.a_log, self.dt_bias, batch, H, G, d, dv, self.taps)
        hybrid.conv_ring(qkv, state["ring"], batch, self.channels, self.taps)
        o = hybrid.recur_scan(rec, v, state["S"], batch, H, d, dv, delta=True)
        hybrid.head_norm_gate(o, self.norm, y, self.eps, gate=gate, mul=scale)


class SSDBranch(Branch):
    """Mamba-2 recurrence (state-space duality): one projection z | x | B | C | dt, a short convolution with bias and silu on x,
    B and C, one decay per head, B and C shared by the heads of a group, output gate silu(z), then an RMS norm in equal
    parts."""

    def __init__(self, heads, vdim, state, groups, taps, norm_parts, eps, dtype=None, device=None):
        super().__init__()
        if heads % groups or (heads * vdim) % norm_parts:
            raise ValueError(f"{heads} heads of size {vdim} do not divide into {groups} groups and {norm_parts} norm parts")
        self.H, self.P, self.N, self.G, self.taps, self.parts, self.eps = heads, vdim, state, groups, taps, norm_parts, eps
        inner = heads * vdim
        self.channels = inner + 2 * groups * state
        self.segments = OrderedDict([("in", inner + self.channels + heads)])
        self.out_width = inner
        f32 = dict(dtype=torch.float32, device=device)
        self.conv = _param(taps, self.channels, fill=1.0 / taps, **f32)
        self.conv_bias = _param(self.channels, **f32)
        self.dt_bias = _param(heads, fill=-2.0, **f32)
        self.a_log = _param(heads, **f32)
        self.skip = _param(heads, fill=1.0, **f32)
        self.norm = _param(inner, fill=1.0, **f32)

    def state_spec(self, act_dtype):
        return {"S": ((self.H, self.N, self.P), torch.float32), "ring": ((self.taps, self.channels), act_dtype)}

    def tensors(self):
        return [("conv", self.conv.data.t()), ("conv.b", self.conv_bias), ("dt_bias", self.dt_bias), ("A_log", self.a_log), ("D", self.skip),
                ("norm", self.norm)]

    def run(self, u, y, batch, state, kv, scale):
        if scale != 1.0:
            raise NotImplementedError("the norm of this branch takes no scale")
        fn = hybrid.ssd_step if batch.decode else hybrid.ssd_prompt
        fn(u["in"], self.conv, self.conv_bias, state["ring"], self.dt_bias, self.a_log, self.skip, state["S"], y, batch, self.H, self.P, self.N,
           self.G, self.taps)
        hybrid.part_rmsnorm_(y, self.norm, self.parts, self.eps)


def rotary_frequencies(dims, base, scaling=None):
    """Angles per position of the ``dims / 2`` rotation pairs (float64) and the factor on cos and sin. ``scaling`` (YaRN:
    factor, original, fast, slow) divides the slow pairs by the factor, leaves the fast ones, and blends in between."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = float(base) ** (-2.0 * i / max(dims, 1))
    if not scaling:
        return f, 1.0

    def pair_of(turns):       # pair that turns this often over the original length
        return dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo, hi = max(math.floor(pair_of(scaling["fast"])), 0), min(math.ceil(pair_of(scaling["slow"])), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0, 1)
    return f * (ramp / scaling["factor"] + (1 - ramp)), 0.1 * math.log(scaling["factor"]) + 1


class PooledAttentionBranch(Branch):
    """Grouped-query attention to a window of tokens and to averages of older blocks (``window``), with projection biases,
    rotated queries and keys, values rotated by their position and turned back by the query's, a temperature per head, a sink
    in the softmax and an elementwise output gate. ``interleaved``: rotation pairs are neighbours instead of halves."""

    def __init__(self, heads, kv_heads, dim, vdim, window, rot_dims, rot_base, scale, scaling=None, interleaved=False, dtype=None, device=None):
        super().__init__()
        if vdim % 2 or rot_dims % 2 or rot_dims > dim:
            raise ValueError(f"rotation of {rot_dims} of {dim} key entries and {vdim} value entries")
        if window.size < 1 or window.pool < 1:
            raise ValueError(f"window of {window.size} tokens with blocks of {window.pool}")
        self.H, self.G, self.d, self.dv, self.window, self.scale, self.interleaved = heads, kv_heads, dim, vdim, window, scale, interleaved
        self.segments = OrderedDict(q=heads * dim, k=kv_heads * dim, v=kv_heads * vdim, g=heads * vdim)
        self.tight = ("q", "k", "v")
        self.out_width = heads * vdim
        f32 = dict(dtype=torch.float32, device=device)
        self.bias = _param(heads * dim + kv_heads * (dim + vdim), **f32)
        self.temp = _param(heads, fill=1.0, **f32)
        self.sink = _param(heads, **f32)
        freq, self.rot_mul = rotary_frequencies(rot_dims, rot_base, scaling)
        self._freq = (freq, rotary_frequencies(vdim, rot_base)[0])

    def freqs(self, device):
        if self._freq[0].device != device:
            self._freq = tuple(f.to(device) for f in self._freq)
        return self._freq

    def kv_spec(self):
        return self.G, self.d, self.dv, self.window

    def tensors(self):
        a, b = self.H * self.d, (self.H + self.G) * self.d
        c = self.bias.data
        return [("q.b", c[:a]), ("k.b", c[a:b]), ("v.b", c[b:]), ("temp", self.temp), ("sink", self.sink)]

    def run(self, u, y, batch, state, kv, scale):
        if scale != 1.0:
            raise NotImplementedError("the gate of this branch takes no scale")
        H, G, d, dv, win = self.H, self.G, self.d, self.dv, self.window
        k_cache, v_cache = kv
        qkv, gate = u["q"], u["g"]
        dev, act = qkv.device, qkv.dtype
        prep = (qkv, self.bias, *self.freqs(dev), self.rot_mul, self.temp, batch, k_cache, v_cache, H, G, d, dv, self.interleaved)
        tc = (hybrid.window_decode_tc if batch.decode else hybrid.window_tc)(act, H, G, d, dv)
        q = dict(q=torch.empty(batch.T, H, _up(d, 16 if batch.decode else 64), dtype=act, device=dev)) if tc else             dict(q32=torch.empty(batch.T, H, d, dtype=torch.float32, device=dev))
        if batch.decode:
            turn = hybrid.win_prep(*prep, **q, pool=win.pool)
            hybrid.window_decode(k_cache, v_cache, self.sink, turn, gate, y, batch, self.scale, H, G, d, dv, win, self.interleaved, **q)
            return
        view = batch.views[win]
        dp, dvp = _up(d), _up(dv)
        k = (torch.empty if dp == d else torch.zeros)(view.rows, G * dp, dtype=act, device=dev)
        v = (torch.empty if dvp == dv else torch.zeros)(view.rows, G * dvp, dtype=act, device=dev)
        # before the append: the append may reuse blocks that earlier positions still occupy
        hybrid.kv_gather(k_cache, view.gather_entry, view.gather_row, k, G, d, dp)
        hybrid.kv_gather(v_cache, view.gather_entry, view.gather_row, v, G, dv, dvp)
        turn = hybrid.win_prep(*prep, **q, k_out=k, v_out=v, dp=dp, dvp=dvp, kv_row=view.kv_row)
        hybrid.pool_blocks(k, dp, k_cache, view, G, d, win.pool)
        hybrid.pool_blocks(v, dvp, v_cache, view, G, dv, win.pool)
        hybrid.window_attention(k, v, dp, dvp, self.sink, turn, gate, y, batch, view, self.scale, H, G, d, dv, win, self.interleaved, **q)


class TalkingAttentionBranch(Branch):
    """Grouped-query attention inside chunks of ``chunk`` positions: short convolutions, query / key norm, interleaved
    rotation, a head mix between scores and softmax, one output gate per head."""

    def __init__(self, heads, kv_heads, dim, vdim, taps, chunk, rot_dims, rot_base, scale, eps, dtype=None, device=None):
        super().__init__()
        self.H, self.G, self.d, self.dv, self.taps, self.eps = heads, kv_heads, dim, vdim, taps, eps
        self.chunk, self.scale, self.rot_dims, self.rot_base = chunk, scale, rot_dims, rot_base
        self.segments = OrderedDict(q=heads * dim, k=kv_heads * dim, v=kv_heads * vdim, g=heads)
        self.tight = ("q", "k", "v")
        self.out_width = heads * vdim
        self.channels = heads * dim + kv_heads * (dim + vdim)
        f32 = dict(dtype=torch.float32, device=device)
        self.conv = _param(taps, self.channels, fill=1.0 / taps, **f32)
        self.q_norm = _param(dim, fill=1.0, **f32)
        self.k_norm = _param(dim, fill=1.0, **f32)
        self.talk = tnn.Parameter(torch.eye(heads, **f32), requires_grad=False)
        i = torch.arange(rot_dims // 2, dtype=torch.float64)
        self._inv = (float(rot_base) ** (-2.0 * i / max(rot_dims, 1)))

    def inv_freq(self, device):
        if self._inv.device != device:
            self._inv = self._inv.to(device)
        return self._inv

    def kv_spec(self):
        return self.G, self.d, self.dv, self.chunk

    def state_spec(self, act_dtype):
        return {"ring": ((self.taps, self.channels), act_dtype)}

    def tensors(self):
        a, b = self.H * self.d, (self.H + self.G) * self.d
        c = self.conv.data
        return [("q.norm", self.q_norm), ("k.norm", self.k_norm), ("q.conv", c[:, :a].t()), ("k.conv", c[:, a:b].t()),
                ("v.conv", c[:, b:].t()), ("talk", self.talk)]

    def run(self, u, y, batch, state, kv, scale):
        H, G, d, dv = self.H, self.G, self.d, self.dv
        k_cache, v_cache = kv
        qkv, gate = u["q"], u["g"]
        dev, act = qkv.device, qkv.dtype
        common = (qkv, self.conv, state["ring"], self.q_norm, self.k_norm, self.inv_freq(dev), batch, k_cache, v_cache, H, G, d, dv,
                  self.taps, self.eps)
        if batch.decode:
            q = qmix = None
            if hybrid.talking_decode_tc(act, H, G, d, dv):
                qmix = torch.empty(batch.T, H, _up(G * d, 64), dtype=act, device=dev)
            else:
                q = torch.empty(batch.T, H, d, dtype=torch.float32, device=dev)
            hybrid.qkv_prep(*common, q_out=q, qmix_out=qmix, talk=self.talk)
            hybrid.talking_decode(q, k_cache, v_cache, self.talk, gate, y, batch, self.scale, scale, H, G, d, dv, self.chunk, qmix=qmix)
            return
        view = batch.views[self.chunk]
        dvp = _up(dv)
        k = torch.empty(view.rows, _up(G * d), dtype=act, device=dev)
        v = torch.empty(view.rows, G * dvp, dtype=act, device=dev)
        # before the append: the append may reuse blocks that earlier positions still occupy
        hybrid.kv_gather(k_cache, view.gather_entry, view.gather_row, k, G, d, d)
        hybrid.kv_gather(v_cache, view.gather_entry, view.gather_row, v, G, dv, dvp)
        if hybrid.talking_tc(act, H, G, d, dv):
            qmix = torch.empty(batch.T, H, _up(G * d, 64), dtype=act, device=dev)
            hybrid.qkv_prep(*common, qmix_out=qmix, talk=self.talk, k_out=k, v_out=v, dvp=dvp, kv_row=view.kv_row)
            hybrid.conv_ring(qkv, state["ring"], batch, self.channels, self.taps)
            hybrid.talking_attention_tc(qmix, k, v, gate, y, batch, view, self.scale, scale, H, G, d, dv, dvp, self.chunk)
            return
        q = torch.empty(batch.T, H, d, dtype=torch.float32, device=dev)
        hybrid.qkv_prep(*common, q_out=q, k_out=k, v_out=v, dvp=dvp, kv_row=view.kv_row)
        hybrid.conv_ring(qkv, state["ring"], batch, self.channels, self.taps)
        hybrid.talking_attention(q, k, v, self.talk, gate, y, batch, view.kv_base, self.scale, scale, H, G, d, dv, dvp, self.chunk)


class _Slices:
    """Column slices of the fused projection of one branch."""

    def __init__(self, u, where, branch):
        self.u, self.where, self.branch = u, where, branch
        tight = getattr(branch, "tight", ())
        self.joint = sum(branch.segments[n] for n in tight) if tight else 0

    def __getitem__(self, name):
        a = self.where[name]
        tight = getattr(self.branch, "tight", ())
        if tight and name == tight[0]:       # the convolved projections are read as one block of columns
            return self.u[:, a: a + self.joint]
        return self.u[:, a: a + self.branch.segments[name]]

    def span(self, first, last, width):
        return self.u[:, self.where[first]: self.where[first] + width]


class FusedMixer(Module):
    """Branches side by side over one input: ``residual += sum_i scale_i * branch_i(h)``."""

    def __init__(self, width, branches: "OrderedDict[str, Tuple[Branch, float]]", dtype=None, device=None, init_std=0.02):
        super().__init__()
        self.prefixes = list(branches)
        self.branches = tnn.ModuleList([b for b, _ in branches.values()])
        self.scales = [float(s) for _, s in branches.values()]
        self.where, off = [], 0
        for b in self.branches:
            w = {}
            for name, rows in b.segments.items():
                w[name] = off
                # segments of a convolved block are adjacent; every other one starts on a 16-byte boundary
                tight = getattr(b, "tight", ())
                off = off + rows if name in tight[:-1] else _up(off + rows)
            self.where.append(w)
        self.in_proj = _param(off, width, dtype=dtype, device=device)
        self.out_cols, c = [], 0
        for b in self.branches:
            self.out_cols.append(c)
            c = _up(c + b.out_width)
        self.out_proj = _param(width, c, dtype=dtype, device=device)
        self._pad_cols = c != sum(b.out_width for b in self.branches)
        if init_std:
            for name, t in self.tensors():
                if t.dim() == 2 and t.shape[1] == width or name.endswith("o"):
                    tnn.init.normal_(t, std=init_std)

    def tensors(self) -> "List[Tuple[str, torch.Tensor]]":
        out = []
        for pre, b, w, c in zip(self.prefixes, self.branches, self.where, self.out_cols):
            out += [(pre + n, self.in_proj.data[w[n]: w[n] + rows]) for n, rows in b.segments.items()]
            out += [(pre + n, t.data if isinstance(t, tnn.Parameter) else t) for n, t in b.tensors()]
            out.append((pre + "o", self.out_proj.data[:, c: c + b.out_width]))
        return out

    def kv_specs(self):
        return [s for s in (b.kv_spec() for b in self.branches) if s is not None]

    def state_spec(self, act_dtype):
        return {pre + k: v for pre, b in zip(self.prefixes, self.branches) for k, v in b.state_spec(act_dtype).items()}

    def forward(self, h, residual, batch: RaggedBatch, state, kvs):
        """h [T, width] activations; adds to ``residual`` (fp32) in place."""
        u = gemm(h, self.in_proj)
        K = self.out_proj.shape[1]
        y = (torch.zeros if self._pad_cols else torch.empty)(batch.T, K, dtype=h.dtype, device=h.device)
        kvs = iter(kvs)
        for pre, b, w, c, s in zip(self.prefixes, self.branches, self.where, self.out_cols, self.scales):
            b.run(_Slices(u, w, b), y[:, c: c + b.out_width], batch, {k[len(pre):]: v for k, v in state.items() if k.startswith(pre)},
                  next(kvs) if b.kv_spec() is not None else None, s)
        gemm(y, self.out_proj, c=residual, beta=1.0, out=residual)
