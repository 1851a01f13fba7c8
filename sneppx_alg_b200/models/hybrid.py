"""Base of the hybrid decoders: a pre-norm stack whose layers each choose a token mixer (recurrence, attention of bounded
reach, or several side by side, ``nn/mixers.py``) and a feed-forward or none. The residual stream is fp32.

The models run on ragged batches (``step``): portions of several sequences at once, from the state that earlier portions
left in a ``serving.kv_cache.HybridCache``. ``forward`` offers the framework's generation interface on top of it.

A family names its mixers (``mixer_types``: type in the layer specification -> factory), its norm and its feed-forward
activation. ``layer_specs`` of the configuration lists the layers: ``type``, ``mixer`` (its sizes) and ``mlp`` (or None).
"""
from __future__ import annotations

import torch
import torch.nn as tnn

from ..nn.decoder_parts import DenseMLP, ResidualRMSNorm
from ..nn.mixers import _param
from ..nn.modules import Module
from ..ops import hybrid
from ..ops.gemm import SoftCap, gemm
from ..ops.ragged import RaggedBatch, as_mask
from .config import ModelConfig


def pick(spec, *names):
    """The named entries of a mixer specification."""
    try:
        return [spec[n] for n in names]
    except KeyError as e:
        raise ValueError(f"layer configuration has no {e.args[0]!r}: {spec}") from None


class HybridLayer(Module):
    def __init__(self, family, cfg: ModelConfig, spec: dict, dtype=None, device=None):
        super().__init__()
        d, kw = cfg.hidden_size, dict(dtype=dtype, device=device)
        if spec["type"] not in family.mixer_types:
            raise ValueError(f"unknown mixer type '{spec['type']}'; known: {sorted(family.mixer_types)}")
        self.norm1 = family.norm_type(d, family.norm_eps(cfg), device=device)
        self.mixer = family.mixer_types[spec["type"]](d, spec["mixer"], family.norm_eps(cfg), kw)
        mlp = spec.get("mlp")
        self.mlp = self.norm2 = None
        if mlp is not None:
            if mlp["kind"] != "dense":
                raise ValueError(f"unknown feed-forward kind '{mlp['kind']}'")
            self.norm2 = family.norm_type(d, family.norm_eps(cfg), device=device)
            self.mlp = DenseMLP(d, mlp["ff"], family.mlp_act, **kw)

    def tensors(self):
        parts = [("norm1", self.norm1), ("mix.", self.mixer)]
        if self.mlp is not None:
            parts[1:1] = [("norm2", self.norm2)]
            parts.append(("mlp.", self.mlp))
        return [(p + n, t) for p, m in parts for n, t in m.tensors()]

    def forward(self, x, batch, act_dtype, state, kvs):
        self.mixer(self.norm1(x, act_dtype), x, batch, state, kvs)
        if self.mlp is not None:
            self.mlp(self.norm2(x, act_dtype), x)


class HybridDecoder(Module):
    mixer_types: dict = {}
    norm_type = ResidualRMSNorm
    mlp_act = "xielu"

    @staticmethod
    def norm_eps(cfg: ModelConfig) -> float:
        return cfg.rms_norm_eps

    def __init__(self, cfg: ModelConfig, dtype=None, device=None):
        super().__init__()
        self.config = cfg
        dtype = dtype or torch.get_default_dtype()
        kw = dict(dtype=dtype, device=device)
        self.embed = _param(cfg.vocab_size, cfg.hidden_size, std=cfg.initializer_range, **kw)
        self.layers = tnn.ModuleList([HybridLayer(type(self), cfg, s, **kw) for s in cfg.layer_specs])
        self.norm = self.norm_type(cfg.hidden_size, self.norm_eps(cfg), device=device)
        self.head = None if cfg.tie_word_embeddings else _param(cfg.vocab_size, cfg.hidden_size, std=cfg.initializer_range, **kw)
        self._cap = SoftCap(cfg.logit_softcap) if cfg.logit_softcap else None

    # ------------------------------------------------------------------ configuration and weights
    @staticmethod
    def config_from_tensors(cfg: ModelConfig, tensors) -> ModelConfig:
        """Sizes that only the tensors give."""
        return cfg

    def tensors(self):
        out = [("embed", self.embed.data)]
        for i, layer in enumerate(self.layers):
            out += [(f"l{i}.{n}", t) for n, t in layer.tensors()]
        out += [("final.norm" + n, t) for n, t in self.norm.tensors()]
        return out + ([("head", self.head.data)] if self.head is not None else [])

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
                layer.mlp.reloaded()
        if missing:
            raise KeyError(f"missing tensors: {missing[:5]}{'...' if len(missing) > 5 else ''}")
        return missing

    # ------------------------------------------------------------------ serving
    @property
    def act_dtype(self):
        return self.embed.dtype

    def init_cache(self, max_sequences, num_blocks=None, block_size=16, max_tokens=None):
        """Block pool and state slots for ``max_sequences`` live sequences. Without ``num_blocks`` there is room for all of
        them; attention that keeps averages of older positions takes it for ``max_tokens`` tokens each (default: the
        configuration's longest sequence, 8192 if it has none)."""
        from ..serving.kv_cache import HybridCache
        specs = [s for layer in self.layers for s in layer.mixer.kv_specs()]
        masks = [s[3] for s in specs]
        if num_blocks is None:
            rules = [as_mask(m) for m in masks]
            each = (max(r.span for r in rules) + block_size - 2) // block_size + 1 if rules else 0
            n = max_tokens or self.config.max_position_embeddings or 8192
            each += sum((n // p + block_size - 1) // block_size for p in {r.pool for r in rules if r.pool})
            num_blocks = max(1, max_sequences * each)
        return HybridCache([s[:3] for s in specs], masks, [layer.mixer.state_spec(self.act_dtype) for layer in self.layers],
                           max_sequences, num_blocks, block_size, self.act_dtype, self.embed.device)

    @torch.no_grad()
    def step(self, batch: RaggedBatch, cache):
        """Runs the rows of a batch from the cache's state and returns fp32 logits of the wanted rows."""
        x = hybrid.embed_f32(self.embed, batch.ids, self.config.embedding_scale)
        kv = 0
        for i, layer in enumerate(self.layers):
            n = len(layer.mixer.kv_specs())
            layer(x, batch, self.act_dtype, cache.state[i], [(cache.k[j], cache.v[j]) for j in range(kv, kv + n)])
            kv += n
        h = self.norm(x, self.act_dtype, rows=batch.want)
        return gemm(h, self.embed if self.head is None else self.head, out_dtype=torch.float32, act=self._cap)

    # ------------------------------------------------------------------ generation interface
    def forward(self, input_ids, attention_mask=None, position_ids=None, past_key_values=None, use_cache=False, labels=None,
                shift_labels=True):
        from ..serving.hybrid_runner import HybridRunner
        B, S = input_ids.shape
        runner = past_key_values
        if runner is None:
            runner = HybridRunner(self, self.init_cache(B, max_tokens=max(S, self.config.max_position_embeddings or 8192)))
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
