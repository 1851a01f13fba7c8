"""Tibalorn decoder: a hybrid stack (``models/hybrid.py``) whose layers each choose a Mamba-2 recurrence (``mamba2``) or
sliding-window attention over tokens and averaged blocks of older tokens (``attention``: YaRN rotation, rotated values,
softmax with a sink, per-head temperature, output gate), with layer norms, a squared-ReLU feed-forward or none, a scaled
embedding that is also the output matrix, and soft-capped logits.

Configuration keys of the checkpoint's ``config.json`` (``architecture: "Tibalorn"``): ``vocab``, ``width``, ``norm.eps``,
``embedding.scale``, ``logit_softcap`` and ``layers``, one entry per layer with ``type``, ``mixer`` and ``mlp``.
"""
from __future__ import annotations

from collections import OrderedDict

from ..nn.decoder_parts import ResidualLayerNorm
from ..nn.mixers import FusedMixer, PooledAttentionBranch, SSDBranch
from ..ops.ragged import PooledWindow
from .config import ModelConfig
from .hybrid import HybridDecoder, pick


def _mamba2(width, m, eps, kw):
    heads, vdim, state, groups, taps, parts = pick(m, "heads", "vdim", "state", "groups", "conv", "norm_groups")
    return FusedMixer(width, OrderedDict([("", (SSDBranch(heads, vdim, state, groups, taps, parts, eps, **kw), 1.0))]), **kw)


def _attention(width, m, eps, kw):
    heads, kv, dim, vdim, mask, rot, scale = pick(m, "heads", "kv_heads", "dim", "vdim", "mask", "rot", "scale")
    window = PooledWindow(*pick(mask, "size", "pool"))
    branch = PooledAttentionBranch(heads, kv, dim, vdim, window, rot["dims"], rot["base"], scale, scaling=rot.get("scaling"), **kw)
    return FusedMixer(width, OrderedDict([("", (branch, 1.0))]), **kw)


class TibalornForCausalLM(HybridDecoder):
    mixer_types = {"mamba2": _mamba2, "attention": _attention}
    norm_type = ResidualLayerNorm
    mlp_act = "relu2"

    @staticmethod
    def norm_eps(cfg: ModelConfig) -> float:
        return cfg.layer_norm_eps
