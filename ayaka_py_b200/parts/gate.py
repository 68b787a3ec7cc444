"""What a sublayer's result passes before it joins the residual stream: a constant per channel and a gate per
channel, sigmoid(W h + b), from the rows h that the sublayer reads.  Where the sublayer's first product can take
another matrix along (``Part.join_input``), the gate's product rides in it.  Gate, constant and sum are 32-bit."""

from __future__ import annotations

import torch

from .. import ops
from .base import Part, TensorDecl, register_part


class ResidualGate(Part):
    KIND = "residual_gate"

    def __init__(self, width: int, dtype=torch.float32, device="cuda"):
        self.width, self.dtype = width, dtype
        self.scale = self.weight = self.bias = None
        self.joined = False

    def tensors(self):
        d = self.width
        return {"scale": TensorDecl((d,), "vector"), "weight": TensorDecl((d, d), "matrix"), "bias": TensorDecl((d,), "vector")}

    def ride(self, sublayer: Part) -> None:
        """Lets the gate's product ride in the sublayer's first one, if the sublayer does this."""
        view = sublayer.join_input(self.weight, self.bias)
        if view is not None:
            self.weight, self.joined = view, True

    def gates(self, sublayer: Part, h: torch.Tensor, ctx) -> torch.Tensor:
        """W h + b, float32 [T, width], after the sublayer has run on h."""
        if self.joined:
            return ctx.carry.pop(sublayer)
        return ops.linear(h, self.weight, self.bias, out_dtype=torch.float32)


register_part(ResidualGate.KIND, ResidualGate)
