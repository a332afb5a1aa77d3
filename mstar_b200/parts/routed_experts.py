"""Routed experts feed-forward: a float router chooses ``top`` of ``experts`` small gated
feed-forwards per token; an optional shared one runs for every token and is added.

The router's logits are a product with float output; a kernel turns them into the chosen
experts and their weights (sigmoid or softmax scores, a correction for the choice, groups of
which the best stay eligible, renormalised and scaled or not).  The shared
expert is the dense gated feed-forward's path (one fused gate/up product, one down
product); the routed experts' kernels add its output while they write theirs, times the
sigmoid of a gate a token where it has one (a further row of the router's product).  A few rows
(decoded tokens) each stream the matrices of their experts; many rows (prompt portions)
are sorted by expert on the device and run as tiles on the tensor cores.
"""
from __future__ import annotations

import torch

from .. import ops
from ..weights.names import ParamSpec
from .base import Runtime
from .registry import register_part


class RoutedExperts:
    graph_safe = True       # shapes are fixed by the batch; the choice stays on the device

    @classmethod
    def param_specs(cls, spec) -> dict:
        e, ff, width = spec.num_experts, spec.expert_size, spec.hidden_size
        outputs = e + spec.identity_experts
        # the shared expert's gate is the row after the router's
        out = {"router.weight": ParamSpec((outputs + (1 if spec.shared_gate else 0), width))}
        if spec.choice_bias:
            out["router.correction"] = ParamSpec((outputs,), role="vector", init="zeros")
        if spec.gated:
            out["experts.gate_up.weight"] = ParamSpec((e * 2 * ff, width))
        else:
            out["experts.up.weight"] = ParamSpec((e * ff, width))
        out["experts.down.weight"] = ParamSpec((e * width, ff))
        if spec.shared_size:
            out["shared.gate_up.weight"] = ParamSpec((2 * spec.shared_size, width))
            out["shared.down.weight"] = ParamSpec((width, spec.shared_size))
        return out

    def __init__(self, spec, params: dict, runtime: Runtime):
        if (spec.gated, spec.activation) not in ((True, "silu"), (True, "clamped_swish"),
                                                 (False, "relu2")):
            raise ValueError(f"routed experts with gated={spec.gated} and activation "
                             f"{spec.activation!r} have no kernel (gated silu, gated clamped_swish "
                             "and plain relu2 have)")
        if spec.shared_gate and not spec.shared_size:
            raise ValueError("a gate on the shared expert needs a shared expert")
        clamped = spec.activation == "clamped_swish"
        self.clamp = (spec.limit, spec.swish_alpha) if clamped else None
        self.shared_clamp = {"limit": spec.shared_limit, "alpha": spec.swish_alpha} if clamped else {}
        if spec.identity_experts and spec.scale_input:
            raise ValueError("identity experts go with weights on the experts' outputs")
        if spec.score not in ("sigmoid", "softmax"):
            raise ValueError(f"router score {spec.score!r} is not known (sigmoid, softmax)")
        self.spec = spec
        self.runtime = runtime
        self.router = params["router.weight"]
        self.outputs = spec.num_experts + spec.identity_experts
        if self.router.shape[0] % 8:            # whole 16-byte rows of logits for the product
            pad = -self.router.shape[0] % 8
            self.router = torch.cat([self.router, self.router.new_zeros((pad, spec.hidden_size))])
        self.gate_up = params["experts.gate_up.weight" if spec.gated else "experts.up.weight"]
        self.correction = None
        if spec.choice_bias:
            self.correction = params["router.correction"].float().contiguous()
        self.down = params["experts.down.weight"]
        self.shared_gate_up = params.get("shared.gate_up.weight")
        self.shared_down = params.get("shared.down.weight")

    def forward(self, x, ctx):
        s = self.spec
        logits = ops.linear(x, self.router, out_dtype=torch.float32, static_weights=True)
        shared_gate = logits[:, self.outputs:self.outputs + 1] if s.shared_gate else None
        logits = logits[:, :self.outputs]
        chosen, weight = ops.route_topk(logits, s.top, softmax=s.score == "softmax",
                                        renormalize=s.renormalize, choice_bias=self.correction,
                                        groups=s.groups, renorm_eps=s.renorm_eps,
                                        weight_scale=s.weight_scale)
        shared = None
        if self.shared_gate_up is not None:
            shared = ops.linear(ops.gated_up(x, self.shared_gate_up, static_weights=True,
                                             kind=s.activation, **self.shared_clamp),
                                self.shared_down, static_weights=True)
        return ops.routed_experts(x, self.gate_up, self.down, chosen, weight, s.num_experts,
                                  s.expert_size, s.scale_input, add=shared, gated=s.gated,
                                  identity=s.identity_experts, clamp=self.clamp,
                                  add_gate=shared_gate)


register_part("ffn", "routed_experts", RoutedExperts)
