"""Mixture of experts with a gated shared expert.

Router: z = W_r h in 32-bit; the ``top`` experts with the largest z are chosen and weighted by
the softmax over the chosen z only.  An expert (no biases): g = min(W_gate h, limit),
u = clamp(W_up h, -limit, limit), y = W_down (g sigmoid(1.702 g) (u + 1)).  The output is the
weighted sum of the chosen experts' y plus the shared expert's (same form, sizes and limit of
its own), which runs for every token and is multiplied by sigmoid(w_mix . h), one number per
token.

Variants, all by parameters: ``router="sigmoid_groups"`` chooses by s + correction with s = sigmoid(z)
and a correction per expert (a tensor of the part) among the experts of the ``keep`` best of ``groups``
equal runs of consecutive experts (a run's score: the sum of its two largest ranking scores; the others cannot be
chosen at all), and weights the chosen experts by s over their sum, times ``route_scale``.  ``slope`` and
``plus`` set the activation g sigmoid(slope g) (u + plus); a limit of None clamps nothing (slope 1, plus 0,
no limit: silu(gate) * up).  ``shared_gated`` False: the shared expert is added as it is;
``shared_inner`` 0: there is none.  ``router="softmax_groups"``: s = softmax(z) over all experts, experts ranked by s,
a run's score its largest s, the weights the chosen s as they are, times ``route_scale``.  ``activation``: experts
without a gate, y = W_down act(W_up h) (no shared expert then).  ``router="sigmoid"``: s = sigmoid(z), the ``top``
largest, the weights the chosen s as they are, times ``route_scale``.  ``weigh`` "input": the weight multiplies the
expert's input instead of its output, y = expert(w h); W_gate and W_up are linear, so it is applied to their 32-bit
products, ahead of the activation.

The experts' matrices are kept stacked ([experts, 2 inner, width] with gate over up, and
[experts, width, inner]); a step sorts its (token, choice) pairs by expert on the device and runs
two grouped products over the sorted rows, so nothing about the routing comes back to the host
(``csrc/moe.cu``): on tcgen05 for bfloat16 steps of many pairs (every expert's rows padded to whole
128-row tiles), pair by pair as matrix-vector products for a handful of pairs, on mma.sync or the
FP32 pipes otherwise.  The router and the shared expert's gate, up and mixing row are one dense product."""

from __future__ import annotations

import torch

from .. import ops
from .base import FeedForward, TensorDecl, register_part
from .stacked import StackedInput


class MoE(FeedForward):
    KIND = "moe"
    GATE_SLOPE = 1.702

    def __init__(self, width: int, experts: int, top: int, inner: int, limit: float | None, shared_inner: int,
                 shared_limit: float | None, router: str = "softmax", groups: int = 1, keep: int = 1,
                 route_scale: float = 1.0, slope: float = GATE_SLOPE, plus: float = 1.0, shared_gated: bool = True,
                 activation: str | None = None, weigh: str = "output", dtype=torch.float32, device="cuda"):
        if not 1 <= top <= min(experts, 16):
            raise ValueError(f"top {top} of {experts} experts: the routing kernel picks 1 to 16")
        if router not in ("softmax", "sigmoid", "sigmoid_groups", "softmax_groups"):
            raise ValueError(f"unknown router {router!r}; known: softmax, sigmoid, sigmoid_groups, softmax_groups")
        if weigh not in ("output", "input") or (weigh == "input" and activation is not None):
            raise ValueError(f"weigh {weigh!r}: 'output', or 'input' for experts with a gate")
        if activation is not None and (activation not in ops.ACTIVATIONS or shared_inner):
            raise ValueError(f"experts without a gate take one of {sorted(ops.ACTIVATIONS)} and no shared expert, got {activation!r}")
        if router != "softmax" and not (1 <= keep <= groups <= 32 and experts % groups == 0 and keep * (experts // groups) >= top):
            raise ValueError(f"{experts} experts in {groups} groups (at most 32) of which {keep} are kept cannot give {top} choices")
        self.width, self.experts, self.top, self.inner = width, experts, top, inner
        self.limit = float("inf") if limit is None else float(limit)
        self.shared_inner, self.dtype = shared_inner, dtype
        self.shared_limit = float("inf") if shared_limit is None else float(shared_limit)
        self.router, self.groups, self.keep, self.route_scale = router, int(groups), int(keep), float(route_scale)
        self.slope, self.plus, self.shared_gated = float(slope), float(plus), bool(shared_gated) and shared_inner > 0
        self.activation, self.weigh = activation, weigh
        self.correction = self.stack = self.joined = None
        # many pairs in bfloat16, rows in whole 16-byte pieces: the experts' products run on tcgen05
        self.tensor_cores = dtype == torch.bfloat16 and width % 8 == 0 and inner % 8 == 0

    def tensors(self):
        d, ff, sf = self.width, self.inner, self.shared_inner
        out = {"router_weight": TensorDecl((self.experts, d), "matrix")}
        if self.router == "sigmoid_groups":
            out["correction"] = TensorDecl((self.experts,), "vector")
        if sf:
            out.update({"shared_gate": TensorDecl((sf, d), "matrix"), "shared_up": TensorDecl((sf, d), "matrix"),
                        "shared_down": TensorDecl((d, sf), "matrix")})
        if self.shared_gated:
            out["shared_mix"] = TensorDecl((1, d), "matrix")
        for e in range(self.experts):
            if self.activation is None:
                out[f"gate_{e}"] = TensorDecl((ff, d), "matrix")
            out[f"up_{e}"] = TensorDecl((ff, d), "matrix")
            out[f"down_{e}"] = TensorDecl((d, ff), "matrix")
        return out

    def bind(self, tensors):
        E, d, ff, sf = self.experts, self.width, self.inner, self.shared_inner
        first, gated = tensors["up_0"], self.activation is None
        self.in_weight = torch.empty((E, 2 * ff if gated else ff, d), dtype=first.dtype, device=first.device)
        self.down_weight = torch.empty((E, d, ff), dtype=first.dtype, device=first.device)
        for e in range(E):
            if gated:
                self.in_weight[e, :ff] = tensors[f"gate_{e}"]
            self.in_weight[e, -ff:] = tensors[f"up_{e}"]
            self.down_weight[e] = tensors[f"down_{e}"]
        groups = [[tensors["router_weight"]]]
        if sf:
            groups.append([tensors[name] for name in ("shared_gate", "shared_up", "shared_mix") if name in tensors])
            self.shared_down = tensors["shared_down"]
        self.stack = StackedInput(d, groups)
        self._take_views()
        if "correction" in tensors:
            self.correction = tensors["correction"]
        for e in range(E):                         # per-expert views, as the loader's bookkeeping expects attributes
            if gated:
                setattr(self, f"gate_{e}", self.in_weight[e, :ff])
            setattr(self, f"up_{e}", self.in_weight[e, -ff:])
            setattr(self, f"down_{e}", self.down_weight[e])

    def _take_views(self) -> None:
        self.router_weight = self.stack.views[0]
        if self.shared_inner:
            self.shared_gate, self.shared_up = self.stack.views[1:3]
        if self.shared_gated:
            self.shared_mix = self.stack.views[3]

    def join_input(self, weight, bias):
        """Another matrix rides in the router's product."""
        at = self.stack.join(weight, bias)
        self._take_views()
        self.joined = (at, at + weight.shape[0])
        return self.stack.views[-1]

    def _experts(self, h, ctx):
        """The chosen experts' rows: (float32 rows, row of every pair or None, routing, the stacked product)."""
        pairs = h.shape[0] * self.top
        logits = ops.linear(h, self.stack.weight, self.stack.bias, out_dtype=torch.float32)
        if self.joined is not None:
            ctx.carry[self] = logits[:, self.joined[0]:self.joined[1]]
        scored = None
        if self.router != "softmax":
            scored = {"correction": self.correction, "groups": self.groups, "keep": self.keep, "factor": self.route_scale}
        if self.router == "softmax_groups":
            scored.update(scores="softmax", group_best=1, normalize=False)
        elif self.router == "sigmoid":
            scored.update(normalize=False)
        many = self.tensor_cores and pairs >= ops.MOE_TENSOR_PAIRS
        few = not many and self.tensor_cores and ops.moe_gemv_takes(h, self.in_weight)
        route = ops.moe_route(logits, self.experts, self.top, scored, plan=not many and not few)
        act = self.activation
        glu = (self.limit, self.slope, self.plus)
        early = self.weigh == "input"
        if many:
            picked, rows = ops.moe_experts_tc(h, self.in_weight, self.down_weight, route, *glu, activation=act, weigh_input=early)
            return picked, rows, route, logits
        glu = glu if act is None else None
        if few:
            # a handful of pairs (a step of single tokens): every pair streams its expert's matrices on its own
            hidden = ops.moe_gemv(h, self.in_weight, route, glu=glu, activation=act, weigh_input=early)
            return ops.moe_gemv(hidden, self.down_weight, route, glu=None), None, route, logits            # [T * K, d]
        hidden = ops.moe_gemm(h, self.in_weight, route, glu=glu, out_dtype=self.dtype, activation=act, weigh_input=early)
        return ops.moe_gemm(hidden, self.down_weight, route, glu=None, out_dtype=torch.float32), None, route, logits

    def forward(self, h, residual, ctx):
        """ff(h) (+ residual), float32 [T, width].  h: rows in the compute dtype."""
        picked, rows, route, product = self._experts(h, ctx)
        shared, mix = self._shared(product)
        if shared is None:
            shared = torch.zeros((h.shape[0], self.width), dtype=torch.float32, device=h.device)
        out = ops.moe_combine(picked, route, shared, mix, rows, weighted=self.weigh == "output")
        if residual is not None:
            residual.add_(out)
            return residual
        return out

    def _shared(self, product):
        """The shared expert's float32 rows and the column of their gates' logits; None for what there is not.
        ``product``: the stacked product of the layer's rows."""
        if not self.shared_inner:
            return None, None
        sp = product[:, self.stack.starts[1]:]
        sh = ops.glu_limited(sp, self.shared_inner, self.shared_limit, self.slope, self.dtype, self.plus)
        return ops.linear(sh, self.shared_down, None, out_dtype=torch.float32), sp[:, 2 * self.shared_inner] if self.shared_gated else None

    def forward_rows(self, h, ctx):
        """The chosen experts' rows (and the shared expert's) themselves: their sum is left to the kernel that needs it."""
        picked, rows, route, product = self._experts(h, ctx)
        shared, mix = self._shared(product)
        return ops.PickedRows(picked, route, rows, weighted=self.weigh == "output", shared=shared, mix=mix)


register_part(MoE.KIND, MoE)
