"""Lightning attention: linear attention with a constant decay per head.

Per head, q = silu(W_q h) and k = silu(W_k h) of ``dim`` numbers, v = silu(W_v h) of ``vdim``,

    S_t = lambda_h S_(t-1) + k_t v_t^T,     o_t = S_t^T q_t

(no softmax, no other scale).  The concatenated heads are divided by the root mean square of all of them
together, multiplied by a weight per channel and by sigmoid(W_g h), then projected out.  S (float32) starts at
zero and lives in the request's state slot; decays, state, norm and gate are 32-bit in both dtypes
(``csrc/lightning.cu``).

A step of single tokens, and every step of the 32-bit engine, takes one product for all projections of the input and
walks token by token; portions of prompts in bfloat16 take q, k and v with their activation in the product's epilogue and
go 64 tokens at a time."""

from __future__ import annotations

import torch

from .. import ops
from .base import Mixer, StateNeed, TensorDecl, register_part
from .stacked import StackedInput


class Lightning(Mixer):
    KIND = "lightning"

    def __init__(self, width: int, heads: int, dim: int, vdim: int, decay, eps: float, dtype=torch.float32, device="cuda"):
        decay = [float(x) for x in decay]
        if len(decay) != heads or not all(0.0 <= x <= 1.0 for x in decay):
            raise ValueError(f"{heads} heads need as many decays from 0 to 1, got {decay}")
        if not 1 <= dim <= 1024:
            raise ValueError(f"heads of {dim} numbers: the kernels take keys of 1 to 1024")
        self.width, self.heads, self.dim, self.vdim, self.decay = width, heads, dim, vdim, decay
        self.eps, self.dtype = float(eps), dtype
        self.stack = self.powers = self.joined = None

    def tensors(self):
        d, hd, hv = self.width, self.heads * self.dim, self.heads * self.vdim
        return {"q_weight": TensorDecl((hd, d), "matrix"), "k_weight": TensorDecl((hd, d), "matrix"),
                "v_weight": TensorDecl((hv, d), "matrix"), "gate_weight": TensorDecl((hv, d), "matrix"),
                "norm": TensorDecl((hv,), "vector"), "out_weight": TensorDecl((d, hv), "matrix")}

    def bind(self, tensors):
        """q | k | v | gate become one product; the decays' powers are made once, in double precision."""
        super().bind(tensors)
        self.stack = StackedInput(self.width, [[self.q_weight, self.k_weight, self.v_weight], [self.gate_weight]])
        self._take_views()
        n = torch.arange(ops.DECAY_CHUNK + 1, dtype=torch.float64)
        powers = torch.tensor(self.decay, dtype=torch.float64)[:, None] ** n[None, :]
        self.powers = powers.to(torch.float32).contiguous().to(self.q_weight.device)

    def _take_views(self) -> None:
        self.q_weight, self.k_weight, self.v_weight, self.gate_weight = self.stack.views[:4]

    def join_input(self, weight, bias):
        at = self.stack.join(weight, bias)
        self._take_views()
        self.joined = (at, at + weight.shape[0])
        return self.stack.views[-1]

    def cache_need(self):
        return StateNeed((self.heads, self.dim, self.vdim), torch.float32)

    def forward(self, h, residual, ctx, cache):
        """residual + mix(h); with ``residual`` None the mixer's output alone, float32 [T, width]."""
        state = ctx.cache.state_layer(cache.group, cache.layer)
        weight, bias, split = self.stack.weight, self.stack.bias, self.stack.starts[1]
        if self.dtype == torch.bfloat16 and ctx.max_q_len > 1 and ops.decay_chunk_takes(self.dim):
            rows = ops.linear(h, weight[:split], None, activation="silu", out_dtype=torch.bfloat16)
            rest = ops.linear(h, weight[split:], None if bias is None else bias[split:], out_dtype=torch.float32)
        else:
            rows = ops.linear(h, weight, bias, out_dtype=torch.float32)
            rest = rows[:, split:]
        raw = ops.decay_recurrence(rows, state, self.powers, ctx, self.heads, self.dim, self.vdim)
        o = ops.rmsnorm_gated(raw, rest[:, :self.heads * self.vdim], self.norm, self.eps, self.dtype)
        if self.joined is not None:
            ctx.carry[self] = rest[:, self.joined[0] - split:self.joined[1] - split]
        return ops.linear(o, self.out_weight, None, residual=residual, out_dtype=torch.float32, out=residual)


register_part(Lightning.KIND, Lightning)
