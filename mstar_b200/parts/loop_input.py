"""What the residual passes before each pass of a looped stretch of layers.

Kind "concat_linear": x becomes ``W [x; x0]``, x0 the embedding output.  With ``W = [W_x |
W_0]`` the second half, ``W_0 x0``, is the same in every pass: it is one product a step, whose
float output becomes the residual of each pass, and ``W_x x`` (float output) stays pending on it
until the pass's first norm adds it.
"""
from __future__ import annotations

import torch

from .. import ops
from ..weights.names import ParamSpec
from .base import ResidualStream, Runtime
from .registry import register_part


class ConcatLinear:
    graph_safe = True       # nothing per-step is read from the host

    @classmethod
    def param_specs(cls, spec) -> dict:
        return {"weight": ParamSpec((spec.hidden_size, 2 * spec.hidden_size))}

    def __init__(self, spec, params: dict, runtime: Runtime):
        self.spec = spec
        self.runtime = runtime
        w = params["weight"]
        # halves with rows of their own: what the products' kernels take
        self.w_x = w[:, :spec.hidden_size].contiguous()
        self.w_0 = w[:, spec.hidden_size:].contiguous()
        self.shared = False     # whether the passes may share one residual tensor

    def begin(self, x0: torch.Tensor) -> torch.Tensor:
        """float ``W_0 x0`` of the step's embedding output."""
        return ops.linear(ops.convert(x0, self.runtime.dtype), self.w_0, out_dtype=torch.float32,
                          static_weights=True)

    def apply(self, stream: ResidualStream, anchor: torch.Tensor) -> None:
        """Put ``W_x x + anchor`` in the residual's place."""
        x = stream.read_rows(self.runtime.dtype)
        stream.take_pending()
        stream.h = anchor if self.shared else anchor.clone()
        stream.push(ops.linear(x, self.w_x, out_dtype=torch.float32, static_weights=True))


register_part("loop_input", "concat_linear", ConcatLinear)
