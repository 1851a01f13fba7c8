"""Rilenex decoder: a hybrid stack (``models/hybrid.py``) whose layers each choose a gated-write recurrence (``hgrn2``) or
chunked talking-heads attention beside a gated delta rule (``parallel``), with RMS norms and an xIELU feed-forward or none.

Configuration keys of the checkpoint's ``config.json`` (``architecture: "Rilenex"``): ``vocab``, ``width``, ``norm.eps`` and
``layers``, one entry per layer with ``type``, ``mixer`` and ``mlp``. The ranks of the low-rank products are only in the
tensors' shapes; ``config_from_tensors`` copies them into the configuration before the model is built.
"""
from __future__ import annotations

import copy
from collections import OrderedDict

from ..nn.mixers import DeltaBranch, FusedMixer, GatedWriteBranch, TalkingAttentionBranch
from .config import ModelConfig
from .hybrid import HybridDecoder, pick


def _hgrn2(width, m, eps, kw):
    heads, dim, vdim = pick(m, "heads", "dim", "vdim")
    return FusedMixer(width, OrderedDict([("", (GatedWriteBranch(heads, dim, vdim, eps, **kw), 1.0))]), **kw)


def _parallel(width, m, eps, kw):
    lt, rt, ls, rs = pick(m, "left", "right", "left_scale", "right_scale")
    heads, kv, dim, vdim, taps, mask, rot, scale = pick(lt, "heads", "kv_heads", "dim", "vdim", "conv", "mask", "rot", "scale")
    left = TalkingAttentionBranch(heads, kv, dim, vdim, taps, mask["size"], rot["dims"], rot["base"], scale, eps, **kw)
    heads, kv, dim, vdim, taps = pick(rt, "heads", "kv_heads", "dim", "vdim", "conv")
    right = DeltaBranch(heads, kv, dim, vdim, taps, rt.get("decay_rank", dim), rt.get("gate_rank", dim), eps, **kw)
    return FusedMixer(width, OrderedDict([("left.", (left, ls)), ("right.", (right, rs))]), **kw)


class RilenexForCausalLM(HybridDecoder):
    mixer_types = {"hgrn2": _hgrn2, "parallel": _parallel}

    @staticmethod
    def config_from_tensors(cfg: ModelConfig, tensors) -> ModelConfig:
        """The ranks of the decay and gate products."""
        cfg.layer_specs = copy.deepcopy(cfg.layer_specs)
        for i, s in enumerate(cfg.layer_specs):
            if s["type"] == "parallel":
                p = f"l{i}.mix.right."
                s["mixer"]["right"]["decay_rank"] = int(tensors[p + "a1"].shape[0])
                s["mixer"]["right"]["gate_rank"] = int(tensors[p + "g1"].shape[0])
        return cfg
