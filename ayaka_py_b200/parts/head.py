"""Logits of the wanted rows: h @ W[:V]^T (times a constant; behind a soft cap c tanh(z / c)), no bias, float32 out
(``models/_common.py:248-253``, ``layers/embedding.py:741-747``)."""

from __future__ import annotations

import torch

from .. import ops
from .base import Head, TensorDecl, register_part


class LMHead(Head):
    KIND = "lm_head"

    def __init__(self, vocab: int, width: int, scale: float = 1.0, softcap: float | None = None,
                 dtype=torch.float32, device="cuda"):
        if softcap is not None and softcap <= 0:
            raise ValueError(f"the logits' cap must be positive, got {softcap}")
        self.vocab, self.width, self.scale, self.softcap = vocab, width, float(scale), softcap
        self.weight = None

    def tensors(self):
        return {"weight": TensorDecl((self.vocab, self.width), "matrix")}

    def forward(self, h, ctx):
        logits = ops.linear(h, self.weight, None, out_dtype=torch.float32)
        if self.scale != 1.0:
            ops.scale_(logits, self.scale)
        return logits if self.softcap is None else ops.softcap_(logits, self.softcap)

    def lower(self, builder, h):
        from ..engine.program import LOGITS
        if self.scale != 1.0 or self.softcap is not None:
            from .base import NotLowered
            raise NotLowered("the step program has no scaled or capped head")
        return builder.linear(h, self.weight, None, out_dtype=torch.float32, out=LOGITS, wanted=True)


register_part(LMHead.KIND, LMHead)
