"""A residual of several streams: what a sublayer reads from them and how its result goes back (hyper-connections)."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..kernels import ops
from ..weights import TensorSpec, MIXING, NORM
from .base import Part


class HyperConnection(Part):
    """One sublayer's connection to n streams: it reads u = sum_s in[s] x_s, and its result y goes back as
    x_t <- sum_s mix[s, t] x_s + out[t] y (`mix` indexed [from, to]). The numbers are kept in 32-bit."""

    def __init__(self, n: int, names: Dict[str, str]):
        super().__init__(names)
        if not 1 <= n <= ops.HYPER_MAX_STREAMS:
            raise ValueError(f"HyperConnection: {n} streams (1..{ops.HYPER_MAX_STREAMS})")
        self.n = int(n)
        self.read = self.write = None          # in [n]; out [n] followed by mix [n * n]

    def local_specs(self):
        return {"in": TensorSpec((self.n,), NORM), "out": TensorSpec((self.n,), NORM), "mix": TensorSpec((self.n, self.n), MIXING)}

    def place(self, local, dtype, device):
        f32 = lambda t: t.to(torch.float32).reshape(-1)
        self.read = f32(local["in"]).to(device).contiguous()
        self.write = torch.cat([f32(local["out"]), f32(local["mix"])]).to(device).contiguous()


class StreamResidual:
    """The streams of one step's tokens while the step runs, 32-bit. At the start all streams are the same rows and only those
    exist; a sublayer's result is not written back at once but kept until something reads the streams, so that the write-back
    of one sublayer and the normed row of the next are one pass over the streams (`ops.hyper_step`), and the last write-back
    and the final norm are one pass over the rows whose logits are wanted."""

    def __init__(self, x0: torch.Tensor, n: int):
        self.n, self.x = n, x0                 # [T, d] (all streams equal) or [n, T, d]
        self.shape = tuple(x0.shape)
        self.waiting: Optional[dict] = None    # a write-back that has not been done: its arguments of `ops.hyper_step`

    def _out(self, ctx):
        return self.x if self.x.dim() == 3 else ctx.empty((self.n,) + self.shape, torch.float32)

    def read(self, ctx, connection: HyperConnection, norm) -> torch.Tensor:
        """The rows that a sublayer reads: norm(sum_s in[s] x_s), in the products' dtype (an RMS norm part)."""
        h = ctx.empty(self.shape)
        if self.waiting is None:
            ops.hyper_step(self.x, self.n, read=connection.read, norm_w=norm.weight, eps=norm.eps, h=h)
            return h
        out = self._out(ctx)
        ops.hyper_step(self.x, self.n, x_out=out, read=connection.read, norm_w=norm.weight, eps=norm.eps, h=h, **self.waiting)
        self.x, self.waiting = out, None
        return h

    def write(self, connection: HyperConnection, y, y_pos=None, y_wts=None, top: int = 1) -> None:
        """A sublayer's result: rows y [T, d], or those of routed pairs (see `RoutedExperts.apply_pairs`)."""
        assert self.waiting is None, "the sublayer before has not been read yet"
        self.waiting = {"write": connection.write, "y": y, "y_pos": y_pos, "y_wts": y_wts, "top": top}

    def total(self, ctx) -> torch.Tensor:
        """The sum of the streams, 32-bit [T, d], as it stands (tests and tools; the engine reads through `final`)."""
        out = ctx.empty(self.shape, torch.float32)
        ops.hyper_step(self.x, self.n, h=out, **(self.waiting or {}))
        return out

    def final(self, ctx, norm, rows: torch.Tensor) -> torch.Tensor:
        """norm(sum of the streams) of the tokens `rows`, in the products' dtype."""
        h = ctx.empty((rows.shape[0], self.shape[1]))
        ops.hyper_step(self.x, self.n, norm_w=norm.weight, eps=norm.eps, h=h, row_idx=rows, **(self.waiting or {}))
        return h
