"""Time mixing (RWKV): a matrix memory per head with a decay per key channel and a bonus for
the current token; the matrix (float) and the last input row live in a state slot.

A kernel makes the five mixes of each token's row with the row before it (and moves the slot's
row on); the products of r, k, v and the gate read a mix each, and with few rows are one launch
together with the decay's first product; a kernel makes the decays (the decay's second product
in it, with few rows) and the current token's weights; the scan walks each entry's tokens from
the matrix in its slot, long portions as pieces side by side; a last kernel norms each head,
scales, gates by ``silu(g)`` and hands the row to the output product.  A prompt portion, a decoded
token and any mix are the same launches.
"""
from __future__ import annotations

from .. import ops
from ..weights.names import ParamSpec
from .base import CacheNeed, LayerCache, Runtime, StateNeed, StepContext
from .registry import register_part


class TimeMixing:
    graph_safe = True       # the forward pass reads the step's device arrays only

    @classmethod
    def param_specs(cls, spec) -> dict:
        rows, width = spec.num_heads * spec.dim, spec.hidden_size
        return {
            # r, k, v, gate and the decay's first product: one launch for few rows
            "in.weight": ParamSpec((4 * rows + spec.decay_rank, width)),
            "mu": ParamSpec((5 * width,), role="vector"),
            "w2.weight": ParamSpec((rows, spec.decay_rank)),
            "w0": ParamSpec((rows,), role="vector", init="zeros"),
            "u": ParamSpec((spec.num_heads, spec.dim), role="vector"),
            "norm.weight": ParamSpec((rows,), role="vector", init="ones"),
            "o.weight": ParamSpec((width, rows)),
        }

    @classmethod
    def cache_need(cls, spec) -> CacheNeed:
        size = ops.time_mixing_state_size(spec.hidden_size, spec.num_heads, spec.dim)
        return CacheNeed(state=StateNeed(shape=(size,), dtype="float32"))

    def __init__(self, spec, params: dict, runtime: Runtime):
        if spec.decay_rank <= 0:
            raise ValueError("the rank of the decay's projection is not known: it comes from the "
                             "checkpoint's tensor shapes or the configuration")
        self.spec = spec
        self.runtime = runtime
        self.w_in = params["in.weight"]
        self.w2 = params["w2.weight"].contiguous()
        self.w_out = params["o.weight"]
        # mixes, decays and bonuses enter the recurrence: float
        self.mu = params["mu"].float().contiguous()
        self.w0 = params["w0"].float().contiguous()
        self.u = params["u"].float().reshape(-1).contiguous()
        self.norm_weight = params["norm.weight"].float().contiguous()

    def forward(self, x, ctx: StepContext, cache: LayerCache):
        s = self.spec
        H, D = s.num_heads, s.dim
        rows = H * D
        mixes = ops.time_mix(x, self.mu, ctx, cache.state)
        rkvg, low = ops.linear_planes(mixes, self.w_in, rows, static_weights=True)
        decay, direct = ops.mix_prepare(rkvg, low, self.w2, self.w0, self.u, H, D, self.runtime.dtype)
        r, k, v, g = (rkvg[:, i * rows:(i + 1) * rows] for i in range(4))
        offset = ops.time_mixing_state_size(s.hidden_size, 0, 0)
        o = ops.linear_scan(r, k, v, decay, direct, ctx, cache.state, offset, H, D, D,
                            vector_decay=True)
        y = ops.head_norm_gate(o, g, self.norm_weight, H, D, s.norm_eps, self.runtime.dtype,
                               kind="silu")
        return ops.linear(y, self.w_out, static_weights=True)


register_part("mixer", "time_mixing", TimeMixing)
