"""Matrices that read the same rows, stacked into one product."""

from __future__ import annotations

import torch


class StackedInput:
    """``groups`` of matrices [n, width]: the matrices of a group lie one under the other, every group starts at a
    multiple of 8 rows (its columns of the product then start on a 16-byte boundary), padding rows are zeros.
    ``join`` adds a group of one matrix.  ``weight`` is the stack, ``bias`` the joined matrices' biases (None
    while there are none), ``starts`` the first row of each group, ``views`` the matrices as views of the stack in
    the order they came."""

    def __init__(self, width: int, groups):
        self.width = width
        self.groups = [list(group) for group in groups]
        self.biases: list[torch.Tensor | None] = [None] * len(self.groups)
        self._build()

    def _build(self) -> None:
        self.starts, rows = [], 0
        for group in self.groups:
            self.starts.append(rows)
            rows += -(-sum(m.shape[0] for m in group) // 8) * 8
        first = self.groups[0][0]
        self.weight = torch.zeros((rows, self.width), dtype=first.dtype, device=first.device)
        self.bias = None
        if any(b is not None for b in self.biases):
            self.bias = torch.zeros((rows,), dtype=torch.float32, device=first.device)
        self.views = []
        for g, group in enumerate(self.groups):
            at = self.starts[g]
            if self.biases[g] is not None:
                self.bias[at:at + self.biases[g].numel()] = self.biases[g]
            for i, m in enumerate(group):
                view = self.weight[at:at + m.shape[0]]
                view.copy_(m)
                group[i] = view
                self.views.append(view)
                at += m.shape[0]

    def join(self, weight: torch.Tensor, bias: torch.Tensor | None) -> int:
        """Adds a group of one matrix; returns the column where its part of the product starts."""
        self.groups.append([weight])
        self.biases.append(bias)
        self._build()
        return self.starts[-1]
