"""Token embedding and output head."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..cache import StateSpec
from ..kernels import ops
from ..weights import TensorSpec, MATRIX
from .base import Part, to_device_matrix
from .linear import linear, EPI_NONE


FUSED_MAX_COLUMNS = 16384


class Embedding(Part):
    """x[t] = table[token[t]] (src/model.br:1286-1295; the reference's embedding scale is 1 here),
    widened to the 32-bit residual stream; `scale` multiplies the rows (in 32-bit)."""

    def __init__(self, vocab: int, dim: int, names: Dict[str, str], scale: float = 1.0):
        super().__init__(names)
        self.vocab, self.dim, self.scale = vocab, dim, float(scale)
        self.table: Optional[torch.Tensor] = None

    def local_specs(self):
        return {"table": TensorSpec((self.vocab, self.dim), MATRIX)}

    def place(self, local, dtype, device):
        self.table = to_device_matrix(local["table"], dtype, device)

    def forward(self, ctx, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        x = ctx.empty((ctx.T, self.dim), torch.float32) if out is None else out
        ops.embed(self.table, ctx.token_ids, x, self.scale)
        return x


class PairEmbedding(Part):
    """x[t] = table[token] + pairs[(previous token * mul_prev + token * mul_cur) mod buckets], 32-bit; a sequence's first token takes
    the row `buckets` of `pairs` [buckets + 1, dim]. The previous token is state of the request: one number in a slot, a cache
    layer of its own that the model numbers behind those of the blocks."""

    def __init__(self, vocab: int, dim: int, buckets: int, mul_prev: int, mul_cur: int, names: Dict[str, str]):
        super().__init__(names)
        self.vocab, self.dim, self.buckets, self.mul_prev, self.mul_cur = vocab, dim, int(buckets), int(mul_prev), int(mul_cur)
        self.table = self.pairs = None

    def local_specs(self):
        return {"table": TensorSpec((self.vocab, self.dim), MATRIX), "pairs": TensorSpec((self.buckets + 1, self.dim), MATRIX)}

    def cache_spec(self):
        return StateSpec((1,), "int32")

    def forward(self, ctx, out: Optional[torch.Tensor] = None, cache_layer: Optional[int] = None) -> torch.Tensor:
        x = ctx.empty((ctx.T, self.dim), torch.float32) if out is None else out
        ops.embed_pairs(self.table, self.pairs, ctx.token_ids, ctx.positions, ctx.tok_req, ctx.cu_q, ctx.slots, ctx.state(cache_layer),
                        self.mul_prev, self.mul_cur, x)
        return x


class OutputHead(Part):
    """logits = y . W^T in 32-bit, no bias (src/model.br:1360-1362). Tied to an embedding: the
    table is shared, not copied (src/model.br:686-690). `softcap` c > 0: logits <- c * tanh(logits / c)."""

    def __init__(self, vocab: int, dim: int, names: Dict[str, str], tied_to: Optional[Embedding] = None, softcap: float = 0.0):
        super().__init__(names)
        self.vocab, self.dim, self.tied_to, self.softcap = vocab, dim, tied_to, float(softcap)
        self.weight: Optional[torch.Tensor] = None

    def local_specs(self):
        return {} if self.tied_to is not None else {"weight": TensorSpec((self.vocab, self.dim), MATRIX)}

    def place(self, local, dtype, device):
        if self.tied_to is None:
            self.weight = to_device_matrix(local["weight"], dtype, device)

    def matrix(self) -> torch.Tensor:
        return self.tied_to.table if self.tied_to is not None else self.weight

    def forward_fused_norm(self, ctx, x: torch.Tensor, norm, row_idx: torch.Tensor) -> Optional[torch.Tensor]:
        """Final norm and output product in one kernel for few rows; None when that is not possible."""
        from .attention import FUSED_MAX_ROWS
        from .norm import RMSNorm
        # every block of the fused kernel normalises the rows again: worth it for a few hundred blocks, not for
        # the thousands that a large vocabulary makes
        if not (ctx.fast and ctx.dtype == torch.bfloat16 and row_idx.shape[0] <= FUSED_MAX_ROWS
                and self.vocab <= FUSED_MAX_COLUMNS
                and isinstance(norm, RMSNorm) and ops.norm_gemm_supported(x, self.matrix())):
            return None
        logits = ctx.empty((row_idx.shape[0], self.vocab), torch.float32)
        ops.norm_gemm(x, norm.weight, norm.eps, self.matrix(), logits, None, EPI_NONE, row_idx)
        if self.softcap > 0:
            ops.softcap(logits, self.softcap)
        return logits

    def forward(self, ctx, y: torch.Tensor) -> torch.Tensor:
        logits = ctx.empty((y.shape[0], self.vocab), torch.float32)
        linear(ctx, y, self.matrix(), logits, None, EPI_NONE)
        if self.softcap > 0:
            ops.softcap(logits, self.softcap)
        return logits
