"""What the next layer reads when it is not simply the stream the last layer left."""
from __future__ import annotations

from typing import Dict

import torch

from ..kernels import ops
from ..weights import TensorSpec, MATRIX, NORM
from .base import Part
from .linear import linear, EPI_NONE


class DepthWeightedAverage(Part):
    """out = sum_{j < n} weight[j] * X_j over the streams so far: X_0 the embedding rows, X_(i+1) what layer i left.
    One such part stands behind every layer (n = i + 2 behind layer i); the sum is 32-bit, in ascending j."""

    def __init__(self, n_inputs: int, names: Dict[str, str]):
        super().__init__(names)
        self.n = int(n_inputs)
        self.weight = None

    def local_specs(self):
        return {"weight": TensorSpec((self.n,), NORM)}

    def forward(self, ctx, streams: torch.Tensor, out: torch.Tensor) -> None:
        ops.depth_mix(streams, self.weight, self.n, out)


class StreamReentry(Part):
    """x <- W [x | x0]: what the first layer of each pass of a loop reads, from the stream x and the embedding rows x0
    (`weight` [dim, 2 dim], x first). The result is a new 32-bit stream; x0 stays as it is."""

    def __init__(self, dim: int, names: Dict[str, str]):
        super().__init__(names)
        self.dim = dim
        self.weight = None

    def local_specs(self):
        return {"weight": TensorSpec((self.dim, 2 * self.dim), MATRIX)}

    def forward(self, ctx, x: torch.Tensor, x0: torch.Tensor) -> torch.Tensor:
        both = ctx.empty((x.shape[0], 2 * self.dim))
        ops.concat_rows(x, x0, both)
        out = ctx.empty(tuple(x.shape), torch.float32)
        after, ctx.next_norm = ctx.next_norm, None       # a fresh stream: no product before it has begun a norm of it
        ctx.memo.pop(("pending norm", id(out)), None)
        linear(ctx, both, self.weight, out, None, EPI_NONE)
        ctx.next_norm = after
        return out


class AfterBlock:
    """What a model with a `DepthWeightedAverage` behind every block wants done once a block has left its stream: the
    average of the streams so far into `out`, and (if the next block begins with a norm) that norm's rows. A block whose
    last kernel works row by row may do both there and set `done`; else the model calls `run_unfused`."""

    def __init__(self, mix: DepthWeightedAverage, streams: torch.Tensor, out: torch.Tensor, next_norm=None):
        self.mix, self.streams, self.out, self.next_norm = mix, streams, out, next_norm
        self.done = False

    def run_unfused(self, ctx) -> None:
        if not self.done:
            self.mix.forward(ctx, self.streams, self.out)
            self.done = True
