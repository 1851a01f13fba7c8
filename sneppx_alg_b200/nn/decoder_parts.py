"""Norms and feed-forwards of the hybrid decoders, whose residual stream is fp32: a norm reads fp32 rows and returns
activations, a feed-forward adds to the residual in its last product's epilogue. Tensor names are those of the checkpoint,
relative to the part (``tensors()``)."""
from __future__ import annotations

from typing import List, Tuple

import torch

from ..ops import hybrid
from ..ops.gemm import XIELU, gemm
from .mixers import _param
from .modules import Module


class ResidualRMSNorm(Module):
    def __init__(self, width, eps, device=None):
        super().__init__()
        self.eps = eps
        self.weight = _param(width, dtype=torch.float32, device=device, fill=1.0)

    def tensors(self) -> "List[Tuple[str, torch.Tensor]]":
        return [("", self.weight.data)]

    def forward(self, x, act_dtype, rows=None):
        return hybrid.rmsnorm_f32(x, self.weight, self.eps, act_dtype, rows=rows)


class ResidualLayerNorm(Module):
    """(x - mean) / sqrt(variance + eps) * weight + bias."""

    def __init__(self, width, eps, device=None):
        super().__init__()
        self.eps = eps
        self.weight = _param(width, dtype=torch.float32, device=device, fill=1.0)
        self.bias = _param(width, dtype=torch.float32, device=device)

    def tensors(self) -> "List[Tuple[str, torch.Tensor]]":
        return [("", self.weight.data), (".b", self.bias.data)]

    def forward(self, x, act_dtype, rows=None):
        return hybrid.layernorm_f32(x, self.weight, self.bias, self.eps, act_dtype, rows=rows)


class DenseMLP(Module):
    """up -> activation (in the GEMM's epilogue) -> down, added to the residual in the second GEMM's epilogue. ``act``: the
    name of a fixed activation, or "xielu" for one with two learned numbers (tensor ``act``)."""

    def __init__(self, width, ff, act, dtype=None, device=None, init_std=0.02):
        super().__init__()
        self.up = _param(ff, width, dtype=dtype, device=device, std=init_std)
        self.down = _param(width, ff, dtype=dtype, device=device, std=init_std)
        self.act = _param(2, dtype=torch.float32, device=device, fill=0.5) if act == "xielu" else None
        self._fixed = None if act == "xielu" else act
        self._fn = None

    def tensors(self) -> "List[Tuple[str, torch.Tensor]]":
        return [("up", self.up.data), ("down", self.down.data)] + ([("act", self.act.data)] if self.act is not None else [])

    def reloaded(self):
        self._fn = None

    def activation(self):
        if self.act is None:
            return self._fixed
        if self._fn is None:
            self._fn = XIELU(*self.act.tolist())
        return self._fn

    def forward(self, h, residual):
        gemm(gemm(h, self.up, act=self.activation()), self.down, c=residual, beta=1.0, out=residual)
