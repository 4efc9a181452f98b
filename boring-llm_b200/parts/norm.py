"""Normalisation parts."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..kernels import ops
from ..weights import TensorSpec, NORM, BIAS
from .base import Part, to_device_vector


class RMSNorm(Part):
    """y = x / sqrt(mean(x^2) + eps) * weight, statistics in 32-bit, the weight used as stored
    (src/math.br:18-36). Input: the 32-bit residual stream; output: the engine's activation dtype.
    `scalar_weight`: the checkpoint holds ONE number (a tensor without dimensions) that multiplies every coordinate; it is
    spread over the width when it is placed, so every kernel that takes an RMS norm's weight takes this one.
    `around_zero`: the checkpoint holds w - 1; the weight 1 + w is formed in 32-bit when it is placed. `gain`: a constant on
    the normed rows, multiplied into the weight in 32-bit when it is placed (a factor on the logits behind a final norm)."""

    def __init__(self, dim: int, eps: float, names: Dict[str, str], scalar_weight: bool = False, around_zero: bool = False,
                 gain: float = 1.0):
        super().__init__(names)
        self.gain = float(gain)
        self.dim, self.eps, self.scalar_weight, self.around_zero = dim, float(eps), bool(scalar_weight), bool(around_zero)
        self.weight: Optional[torch.Tensor] = None

    def local_specs(self):
        return {"weight": TensorSpec(() if self.scalar_weight else (self.dim,), BIAS if self.around_zero else NORM)}

    def place(self, local, dtype, device):
        w = local["weight"]
        if self.scalar_weight:
            w = w.reshape(1).expand(self.dim).contiguous()
        if self.around_zero:
            w = w.to(torch.float32) + 1.0
        if self.gain != 1.0:
            w = w.to(torch.float32) * self.gain
        self.weight = to_device_vector(w, dtype, device)

    def forward(self, ctx, x: torch.Tensor, row_idx: Optional[torch.Tensor] = None, pending_ok: bool = False):
        """The normed rows. `pending_ok`: the caller can finish a norm that the product before it has begun; it then
        gets `PendingNormRows` when the step holds them for this stream and this norm."""
        if pending_ok and row_idx is None:
            held = ctx.memo.get(("pending norm", id(x)))
            if held is not None and held.norm is self:
                return held
        rows = x.shape[0] if row_idx is None else row_idx.shape[0]
        out = ctx.empty((rows, self.dim))
        ops.rmsnorm(x, self.weight, self.eps, out, row_idx)
        return out


class LayerNorm(Part):
    """y = (x - mean) / sqrt(var + eps) * weight + bias over each row, var the mean of the squared deviations; statistics
    in 32-bit. Input: the 32-bit residual stream (or any 32-bit rows); output: the engine's activation dtype.
    `bias=False`: no bias tensor."""

    def __init__(self, dim: int, eps: float, names: Dict[str, str], bias: bool = True):
        super().__init__(names)
        self.dim, self.eps, self.has_bias = dim, float(eps), bool(bias)
        self.weight: Optional[torch.Tensor] = None
        self.bias: Optional[torch.Tensor] = None

    def local_specs(self):
        s = {"weight": TensorSpec((self.dim,), NORM)}
        if self.has_bias:
            s["bias"] = TensorSpec((self.dim,), BIAS)
        return s

    def forward(self, ctx, x: torch.Tensor, row_idx: Optional[torch.Tensor] = None, pending_ok: bool = False):
        rows = x.shape[0] if row_idx is None else row_idx.shape[0]
        out = ctx.empty((rows, self.dim))
        ops.layernorm(x, self.weight, self.bias, self.eps, out, row_idx)
        return out
