"""State-space mixer (Mamba-2): a matrix state per head with one decay a head; the state
(float) and the last inputs of its short convolution live in a state slot.

One product, with float output, gives ``[z | x | B | C | dt]``; a kernel runs the convolution with
bias and SiLU over the x, B and C channels and makes step sizes and decays; the scan walks each
entry's tokens from the state in its slot (long portions as pieces side by side) and moves the
convolution's rows on; a last kernel gates by ``silu(z)``, norms in equal parts and hands the row
to the output product.  A prompt portion, a decoded token and any mix are the same launches.
"""
from __future__ import annotations

import torch

from .. import ops
from ..weights.names import ParamSpec
from .base import CacheNeed, LayerCache, Runtime, StateNeed, StepContext
from .registry import register_part


class StateSpace:
    graph_safe = True       # the forward pass reads the step's device arrays only

    @classmethod
    def param_specs(cls, spec) -> dict:
        inner, channels, heads = spec.inner, spec.channels, spec.num_heads
        return {
            "in.weight": ParamSpec((inner + channels + heads, spec.hidden_size)),
            "conv.weight": ParamSpec((channels, spec.conv), role="vector"),
            "conv.bias": ParamSpec((channels,), role="vector", init="zeros"),
            "dt_bias": ParamSpec((heads,), role="vector", init="zeros"),
            "A_log": ParamSpec((heads,), role="vector", init="zeros"),
            "D": ParamSpec((heads,), role="vector", init="ones"),
            "norm.weight": ParamSpec((inner,), role="vector", init="ones"),
            "o.weight": ParamSpec((spec.hidden_size, inner)),
        }

    @classmethod
    def cache_need(cls, spec) -> CacheNeed:
        size = ops.state_space_state_size(spec.channels, spec.conv, spec.num_heads, spec.state,
                                          spec.v_dim)
        return CacheNeed(state=StateNeed(shape=(size,), dtype="float32"))

    def __init__(self, spec, params: dict, runtime: Runtime):
        if spec.num_heads % spec.groups or spec.inner % spec.norm_groups:
            raise ValueError(f"{spec.num_heads} heads in {spec.groups} groups, {spec.inner} features in "
                             f"{spec.norm_groups} parts do not divide")
        self.spec = spec
        self.runtime = runtime
        self.w_in = params["in.weight"]
        self.w_out = params["o.weight"]
        self.conv_wt = params["conv.weight"].float().t().contiguous()       # taps-major
        self.conv_b = params["conv.bias"].float().contiguous()
        self.dt_bias = params["dt_bias"].float().contiguous()
        self.a_exp = torch.exp(params["A_log"].float()).contiguous()
        self.d_skip = params["D"].float().contiguous()
        self.norm_weight = params["norm.weight"].float().contiguous()

    def forward(self, x, ctx: StepContext, cache: LayerCache):
        s = self.spec
        H, N, VD, inner, channels = s.num_heads, s.state, s.v_dim, s.inner, s.channels
        proj = ops.linear(x, self.w_in, out_dtype=torch.float32, static_weights=True)
        xbc, dt, decay = ops.ssd_prepare(proj, self.conv_wt, self.conv_b, self.dt_bias, self.a_exp,
                                         ctx, cache.state, inner, channels, s.conv, H)
        b, c = xbc[:, inner:inner + s.groups * N], xbc[:, inner + s.groups * N:]
        offset = ops.state_space_state_size(channels, s.conv, 0, 0, 0)
        y = ops.linear_scan(c, b, xbc[:, :inner], decay, self.d_skip, ctx, cache.state, offset, H, N,
                            VD, vector_decay=False, rk_share=H // s.groups, dt=dt,
                            raw=proj[:, inner:], channels=channels, taps=s.conv)
        y = ops.head_norm_gate(y, proj[:, :inner], self.norm_weight, s.norm_groups,
                               inner // s.norm_groups, s.norm_eps, self.runtime.dtype, kind="silu",
                               gate_first=True)
        return ops.linear(y, self.w_out, static_weights=True)


register_part("mixer", "state_space", StateSpace)
