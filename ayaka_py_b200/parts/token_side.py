"""A table's row per token that joins the residual stream at a layer: with e the layer's columns of the token's row,

    y = W_proj (gelu_tanh(W_gate x) * e),     x += y / sqrt(mean(y^2) + eps) * w.

The table is one tensor for all layers (``columns`` wide); a layer reads ``dim`` of them from ``col0`` on.  The gate
reads the stream itself, without a norm: a few rows straight from its 32-bit numbers (a warp per number), many
rows from a copy in the compute dtype that the kernel before leaves.  The norm and the sum are 32-bit."""

from __future__ import annotations

import torch

from .. import ops
from .base import Part, TensorDecl, register_part


class TokenSide(Part):
    KIND = "token_side"

    def __init__(self, vocab: int, width: int, dim: int, columns: int, col0: int, eps: float, dtype=torch.float32, device="cuda"):
        if not 0 <= col0 <= columns - dim:
            raise ValueError(f"columns {col0} .. {col0 + dim - 1} of a table of {columns}")
        self.vocab, self.width, self.dim, self.columns, self.col0 = vocab, width, dim, columns, col0
        self.eps, self.dtype = float(eps), dtype
        self.table = self.gate_weight = self.proj_weight = self.norm = None

    def tensors(self):
        return {"table": TensorDecl((self.vocab, self.columns), "matrix"), "gate_weight": TensorDecl((self.dim, self.width), "matrix"),
                "proj_weight": TensorDecl((self.width, self.dim), "matrix"), "norm": TensorDecl((self.width,), "vector")}

    def reads_copy(self, rows: int) -> bool:
        """Whether ``forward`` wants the stream's rows in the compute dtype as well."""
        return rows > ops.TOKEN_GATE_ROWS and self.dtype != torch.float32

    def forward(self, x: torch.Tensor, copy: torch.Tensor | None, ctx) -> torch.Tensor:
        """y, float32 [T, width]; x: the stream, ``copy``: its rows in the compute dtype (see ``reads_copy``)."""
        if x.shape[0] > ops.TOKEN_GATE_ROWS:
            z = ops.linear(x if copy is None else copy, self.gate_weight, None, out_dtype=torch.float32)
            g = ops.token_gate(ctx.tokens, self.table, self.col0, self.dim, z=z)
        else:
            g = ops.token_gate(ctx.tokens, self.table, self.col0, self.dim, x=x, weight=self.gate_weight)
        return ops.linear(g, self.proj_weight, None, out_dtype=torch.float32)


register_part(TokenSide.KIND, TokenSide)
