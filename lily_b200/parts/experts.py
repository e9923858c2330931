"""A routed mixture of small feed-forward layers, some of whose router outputs may stand for the identity.

The router scores ``s = softmax(W_router h)`` over all its outputs, or each output by itself, ``s = sigmoid(W_router h)``
(logits and scores in float32).  The ``top`` outputs with the largest ``s`` (``+ correction``) are chosen, with ``groups`` only
among those of the ``keep_groups`` best of that many equal runs of neighbouring outputs (a run's score is the sum of its two
largest choice scores); their weights are
their scores ``s`` (without the correction), divided by the sum of the chosen scores where the spec renormalises.  The first
``experts`` outputs name experts with weights of their own,

    y = W_down (g * sigmoid(alpha g) * (u + 1)),   g = min(W_gate h, limit),   u = clamp(W_up h, -limit, limit),

or, with ``activation`` "silu", ``y = W_down (silu(W_gate h) * W_up h)``, or, ungated, with "relu2",
``y = W_down max(W_up h, 0)^2``; the last ``identity`` outputs name experts without
tensors whose output is ``h`` itself.  A weight multiplies the expert's output, or, with ``weight_on`` "input", its input:
``sum_e expert_e(w_e h)``; gate and up products are linear in it, so it is applied to their results ahead of the activation
and one gathered row serves either form.  A shared expert (a feed-forward of the experts' form that every token takes) may
be added, times ``sigmoid(W_sg h)``, one number a token: ``W_sg`` is one more row of the router's product.  The sum is
returned in float32 as one plane of partial sums for the next residual add.

Routing, grouping by expert and the grouped products all stay on the device (``ops.moe_route``, ``ops.moe_experts``):
nothing is read back by the host, so a step replays from a CUDA graph, and each (token, choice) pair is a row of a
grouped product whose sum runs over k in a fixed order, so a token's result does not depend on its neighbours in the
batch.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Optional, Tuple

import torch

from lily_b200.parts.base import BuildContext, FeedForward, TensorSpec, build_part, register_part
from lily_b200.parts.mlp import DenseMLPSpec, SwiGLUSpec


@dataclass(frozen=True)
class RoutedExpertsSpec:
    hidden_size: int
    intermediate_size: int        # of one expert
    experts: int                  # router outputs with weights of their own
    identity: int                 # router outputs after those that stand for the identity
    top: int
    limit: float = 0.0            # "swish_clamped": the clamp on the gate (from above) and on the up product (both sides)
    alpha: float = 1.702          # the slope inside the gate's sigmoid
    scores: str = "softmax"       # "softmax" over all outputs | "sigmoid" of each
    correction: bool = True       # a number an output that is added to its score for the choice alone
    renormalise: bool = True      # the chosen weights are divided by their sum
    activation: str = "swish_clamped"     # of the experts: "swish_clamped" | "silu" | "relu2" (ungated)
    weight_on: str = "output"     # what a weight multiplies: the expert's "output" | its "input"
    shared_size: int = 0          # intermediate size of the shared expert; 0: none
    groups: int = 0               # equal runs of neighbouring outputs of which the best ``keep_groups`` can be chosen from; 0: none
    keep_groups: int = 0
    kind: str = "routed_experts"
    # names under the part's prefix: the router, its correction, the pattern of an expert's prefix, the shared expert's
    # prefix and its gate's row
    names: Optional[Tuple[Tuple[str, str], ...]] = None

    _DEFAULTS = (("router", "router"), ("correction", "correction"), ("expert", "e{}"), ("gate", "gate"), ("up", "up"),
                 ("down", "down"), ("shared", "shared"), ("shared_gate", "shared.sg"))

    def name(self, role: str) -> str:
        return dict(self.names or ()).get(role, dict(self._DEFAULTS)[role])

    @property
    def gated(self) -> bool:
        return self.activation != "relu2"

    @property
    def outputs(self) -> int:
        return self.experts + self.identity


@register_part("feed_forward", "routed_experts")
class RoutedExperts(FeedForward):
    def __init__(self, spec: RoutedExpertsSpec, prefix: str, ctx: BuildContext):
        if spec.experts < 0 or spec.identity < 0 or not 1 <= spec.top <= spec.outputs:
            raise ValueError(f"top {spec.top} of {spec.experts} experts and {spec.identity} identity outputs")
        if spec.scores not in ("softmax", "sigmoid") or spec.activation not in ("swish_clamped", "silu", "relu2") or spec.weight_on not in ("output", "input"):
            raise ValueError(f"routed experts: scores {spec.scores!r}, activation {spec.activation!r}, weight on the {spec.weight_on!r}")
        if spec.weight_on == "input" and spec.identity:
            raise ValueError("a weight on the input has no place in an output that stands for the identity")
        if spec.groups > 1 and (spec.outputs % spec.groups or not 1 <= spec.keep_groups <= spec.groups
                                or spec.top > spec.keep_groups * (spec.outputs // spec.groups)):
            raise ValueError(f"top {spec.top} of the best {spec.keep_groups} of {spec.groups} groups of {spec.outputs} outputs")
        self.spec, self.prefix, self.ctx = spec, prefix, ctx
        self.router = self.correction = self.w_gate_up = self.w_down = None
        self.shared = None
        if spec.shared_size:
            names = tuple((r, spec.name(r)) for r in ("gate", "up", "down"))
            form = SwiGLUSpec(spec.hidden_size, spec.shared_size, names=names) if spec.gated else \
                DenseMLPSpec(spec.hidden_size, spec.shared_size, activation=spec.activation, names=names)
            self.shared = build_part("feed_forward", form, f"{prefix}.{spec.name('shared')}", ctx)
        self.parts = () if self.shared is None else (self.shared,)

    def _expert(self, e: int, role: str) -> str:
        return f"{self.prefix}.{self.spec.name('expert').format(e)}.{self.spec.name(role)}"

    def tensors(self) -> Dict[str, TensorSpec]:
        s, p = self.spec, self.prefix
        out = {f"{p}.{s.name('router')}": TensorSpec((s.outputs, s.hidden_size))}
        if s.correction:
            out[f"{p}.{s.name('correction')}"] = TensorSpec((s.outputs,), role="vector", init="zeros")
        if self.shared is not None:
            out.update(self.shared.tensors())
            out[f"{p}.{s.name('shared_gate')}"] = TensorSpec((1, s.hidden_size))
        for e in range(s.experts):
            if s.gated:
                out[self._expert(e, "gate")] = TensorSpec((s.intermediate_size, s.hidden_size))
            out[self._expert(e, "up")] = TensorSpec((s.intermediate_size, s.hidden_size))
            out[self._expert(e, "down")] = TensorSpec((s.hidden_size, s.intermediate_size))
        return out

    def load(self, get) -> None:
        s, p = self.spec, self.prefix
        # the logits are float32 sums of exact terms either way (a router matrix is served in the compute dtype)
        self.router = get(f"{p}.{s.name('router')}").contiguous()
        if s.correction:
            self.correction = get(f"{p}.{s.name('correction')}").float().contiguous()
        if self.shared is not None:
            self.shared.load(get)
            self.router = torch.cat([self.router, get(f"{p}.{s.name('shared_gate')}")], 0).contiguous()
        if self.router.dtype == torch.bfloat16 and self.router.shape[0] % 8:
            self.router = torch.cat([self.router, self.router.new_zeros(-self.router.shape[0] % 8, s.hidden_size)], 0).contiguous()
        ff, h = s.intermediate_size, s.hidden_size
        if s.experts:
            first = get(self._expert(0, "up"))
            self.w_gate_up = torch.empty((s.experts, 2 * ff if s.gated else ff, h), dtype=first.dtype, device=first.device)
            self.w_down = torch.empty((s.experts, h, ff), dtype=first.dtype, device=first.device)
            for e in range(s.experts):
                if s.gated:
                    self.w_gate_up[e, :ff].copy_(get(self._expert(e, "gate")))
                self.w_gate_up[e, -ff:].copy_(get(self._expert(e, "up")))
                self.w_down[e].copy_(get(self._expert(e, "down")))
        else:
            self.w_gate_up = self.w_down = torch.empty((0,), dtype=self.ctx.dtype, device=self.router.device)

    def forward(self, x, batch):
        s, ops = self.spec, self.ctx.ops
        grouped = {"groups": s.groups, "keep_groups": s.keep_groups} if s.groups > 1 else {}
        routing = ops.moe_route(x, self.router, self.correction, s.top, s.experts, scores=s.scores, renormalise=s.renormalise,
                                shared_gate=self.shared is not None, outputs=s.outputs, **grouped)
        shared = None if self.shared is None else self.shared.forward(x, batch)
        out = ops.moe_experts(x, routing, self.w_gate_up, self.w_down, s.limit, s.alpha, activation=s.activation,
                              weight_on_input=s.weight_on == "input", shared=shared)
        return out.unsqueeze(0)                   # float32 [1, tokens, hidden]: one plane of partial sums
