"""Rilenex decoder: a pre-norm stack whose layers each choose a mixer - a gated-write recurrence (``hgrn2``) or chunked
talking-heads attention beside a gated delta rule (``parallel``) - and an xIELU feed-forward or none. The residual stream
is fp32.

The model runs on ragged batches (``step``): portions of several sequences at once, from the state that earlier portions
left in a ``serving.kv_cache.HybridCache``. ``forward`` offers the framework's generation interface on top of it.

Configuration keys of the checkpoint's ``config.json`` (``architecture: "Rilenex"``): ``vocab``, ``width``, ``norm.eps`` and
``layers``, one entry per layer with ``type``, ``mixer`` and ``mlp``. The ranks of the low-rank products are only in the
tensors' shapes; ``config_from_tensors`` copies them into the configuration before the model is built.
"""
from __future__ import annotations

import copy
from collections import OrderedDict

import torch
import torch.nn as tnn

from ..nn.mixers import DeltaBranch, FusedMixer, GatedWriteBranch, TalkingAttentionBranch, _param
from ..nn.modules import Module
from ..ops import hybrid
from ..ops.gemm import XIELU, gemm
from ..ops.ragged import RaggedBatch
from .config import ModelConfig


def _pick(spec, *names):
    try:
        return [spec[n] for n in names]
    except KeyError as e:
        raise ValueError(f"layer configuration has no {e.args[0]!r}: {spec}") from None


def _hgrn2(width, m, eps, kw):
    heads, dim, vdim = _pick(m, "heads", "dim", "vdim")
    return FusedMixer(width, OrderedDict([("", (GatedWriteBranch(heads, dim, vdim, eps, **kw), 1.0))]), **kw)


def _parallel(width, m, eps, kw):
    lt, rt, ls, rs = _pick(m, "left", "right", "left_scale", "right_scale")
    heads, kv, dim, vdim, taps, mask, rot, scale = _pick(lt, "heads", "kv_heads", "dim", "vdim", "conv", "mask", "rot", "scale")
    left = TalkingAttentionBranch(heads, kv, dim, vdim, taps, mask["size"], rot["dims"], rot["base"], scale, eps, **kw)
    heads, kv, dim, vdim, taps = _pick(rt, "heads", "kv_heads", "dim", "vdim", "conv")
    right = DeltaBranch(heads, kv, dim, vdim, taps, rt.get("decay_rank", dim), rt.get("gate_rank", dim), eps, **kw)
    return FusedMixer(width, OrderedDict([("left.", (left, ls)), ("right.", (right, rs))]), **kw)


MIXER_TYPES = {"hgrn2": _hgrn2, "parallel": _parallel}


class DenseXIELU(Module):
    """up -> xIELU (in the GEMM's epilogue) -> down, added to the residual in the second GEMM's epilogue."""

    def __init__(self, width, ff, dtype=None, device=None, init_std=0.02):
        super().__init__()
        self.up = _param(ff, width, dtype=dtype, device=device, std=init_std)
        self.down = _param(width, ff, dtype=dtype, device=device, std=init_std)
        self.act = _param(2, dtype=torch.float32, device=device, fill=0.5)
        self._fn = None

    def tensors(self):
        return [("up", self.up.data), ("down", self.down.data), ("act", self.act.data)]

    def activation(self):
        if self._fn is None:
            self._fn = XIELU(*self.act.tolist())
        return self._fn

    def forward(self, h, residual):
        gemm(gemm(h, self.up, act=self.activation()), self.down, c=residual, beta=1.0, out=residual)


class RilenexLayer(Module):
    def __init__(self, cfg: ModelConfig, spec: dict, dtype=None, device=None):
        super().__init__()
        d, kw = cfg.hidden_size, dict(dtype=dtype, device=device)
        if spec["type"] not in MIXER_TYPES:
            raise ValueError(f"unknown mixer type '{spec['type']}'; known: {sorted(MIXER_TYPES)}")
        self.eps = cfg.rms_norm_eps
        self.norm1 = _param(d, dtype=torch.float32, device=device, fill=1.0)
        self.mixer = MIXER_TYPES[spec["type"]](d, spec["mixer"], cfg.rms_norm_eps, kw)
        mlp = spec.get("mlp")
        self.mlp = self.norm2 = None
        if mlp is not None:
            if mlp["kind"] != "dense":
                raise ValueError(f"unknown feed-forward kind '{mlp['kind']}'")
            self.norm2 = _param(d, dtype=torch.float32, device=device, fill=1.0)
            self.mlp = DenseXIELU(d, mlp["ff"], **kw)

    def tensors(self):
        out = [("norm1", self.norm1.data)]
        if self.mlp is not None:
            out.append(("norm2", self.norm2.data))
        out += [("mix." + n, t) for n, t in self.mixer.tensors()]
        if self.mlp is not None:
            out += [("mlp." + n, t) for n, t in self.mlp.tensors()]
        return out

    def forward(self, x, batch, act_dtype, state, kvs):
        self.mixer(hybrid.rmsnorm_f32(x, self.norm1, self.eps, act_dtype), x, batch, state, kvs)
        if self.mlp is not None:
            self.mlp(hybrid.rmsnorm_f32(x, self.norm2, self.eps, act_dtype), x)


class RilenexForCausalLM(Module):
    def __init__(self, cfg: ModelConfig, dtype=None, device=None):
        super().__init__()
        self.config = cfg
        dtype = dtype or torch.get_default_dtype()
        kw = dict(dtype=dtype, device=device)
        self.embed = _param(cfg.vocab_size, cfg.hidden_size, std=cfg.initializer_range, **kw)
        self.layers = tnn.ModuleList([RilenexLayer(cfg, s, **kw) for s in cfg.layer_specs])
        self.norm = _param(cfg.hidden_size, dtype=torch.float32, device=device, fill=1.0)
        self.head = _param(cfg.vocab_size, cfg.hidden_size, std=cfg.initializer_range, **kw)

    # ------------------------------------------------------------------ configuration and weights
    @staticmethod
    def config_from_tensors(cfg: ModelConfig, tensors) -> ModelConfig:
        """Sizes that only the tensors give: the ranks of the decay and gate products."""
        cfg.layer_specs = copy.deepcopy(cfg.layer_specs)
        for i, s in enumerate(cfg.layer_specs):
            if s["type"] == "parallel":
                p = f"l{i}.mix.right."
                s["mixer"]["right"]["decay_rank"] = int(tensors[p + "a1"].shape[0])
                s["mixer"]["right"]["gate_rank"] = int(tensors[p + "g1"].shape[0])
        return cfg

    def tensors(self):
        out = [("embed", self.embed.data)]
        for i, layer in enumerate(self.layers):
            out += [(f"l{i}.{n}", t) for n, t in layer.tensors()]
        return out + [("final.norm", self.norm.data), ("head", self.head.data)]

    def to_reference_state_dict(self):
        """Tensors under their checkpoint names."""
        return {n: t.detach().clone().contiguous() for n, t in self.tensors()}

    @torch.no_grad()
    def load_reference_state_dict(self, sd, strict=True):
        missing = []
        for name, dst in self.tensors():
            if name not in sd:
                missing.append(name)
                continue
            src = torch.as_tensor(sd[name])
            if tuple(src.shape) != tuple(dst.shape):
                raise ValueError(f"{name}: checkpoint shape {tuple(src.shape)}, model shape {tuple(dst.shape)}")
            dst.copy_(src)
        for layer in self.layers:
            if layer.mlp is not None:
                layer.mlp._fn = None
        if missing:
            raise KeyError(f"missing tensors: {missing[:5]}{'...' if len(missing) > 5 else ''}")
        return missing

    # ------------------------------------------------------------------ serving
    @property
    def act_dtype(self):
        return self.embed.dtype

    def init_cache(self, max_sequences, num_blocks=None, block_size=16):
        """Block pool and state slots for ``max_sequences`` live sequences (``num_blocks``: default room for all of them)."""
        from ..serving.kv_cache import HybridCache
        specs = [s for layer in self.layers for s in layer.mixer.kv_specs()]
        sizes = [s[3] for s in specs]
        if num_blocks is None:
            num_blocks = max_sequences * ((max(sizes) + block_size - 2) // block_size + 1) if sizes else 1
        return HybridCache([s[:3] for s in specs], sizes, [layer.mixer.state_spec(self.act_dtype) for layer in self.layers],
                           max_sequences, num_blocks, block_size, self.act_dtype, self.embed.device)

    @torch.no_grad()
    def step(self, batch: RaggedBatch, cache):
        """Runs the rows of a batch from the cache's state and returns fp32 logits of the wanted rows."""
        x = hybrid.embed_f32(self.embed, batch.ids)
        kv = 0
        for i, layer in enumerate(self.layers):
            n = len(layer.mixer.kv_specs())
            layer(x, batch, self.act_dtype, cache.state[i], [(cache.k[j], cache.v[j]) for j in range(kv, kv + n)])
            kv += n
        h = hybrid.rmsnorm_f32(x, self.norm, self.config.rms_norm_eps, self.act_dtype, rows=batch.want)
        return gemm(h, self.head, out_dtype=torch.float32)

    # ------------------------------------------------------------------ generation interface
    def forward(self, input_ids, attention_mask=None, position_ids=None, past_key_values=None, use_cache=False, labels=None,
                shift_labels=True):
        from ..serving.hybrid_runner import HybridRunner
        B, S = input_ids.shape
        runner = past_key_values
        if runner is None:
            runner = HybridRunner(self, self.init_cache(B))
            for b in range(B):
                runner.cache.add_sequence(b)
        rows = input_ids.tolist()
        logits = runner.step([(b, rows[b], range(S)) for b in range(B)]).view(B, S, -1)
        out = {"past_key_values": runner if use_cache else None, "logits": logits}
        if labels is not None:
            tgt = labels
            if shift_labels:
                tgt = torch.full_like(labels, -100)
                tgt[:, :-1] = labels[:, 1:]
            out["loss"] = torch.nn.functional.cross_entropy(logits.flatten(0, 1), tgt.flatten(), ignore_index=-100)
        return out
