"""Linear attention over shifted rows, with a decay per head and key channel made from the input and a
bonus for the current token (the formulas are with :class:`TimeMixingSpec`).

``ops.token_blend`` makes the five blends of every row with the row before it (the last row of a
portion is per-request state); one batched product makes r, k, v and the gate from four of them;
two small products with a tanh between make the decay's argument from the fifth, the second with
32-bit output, as it enters the recurrence.  ``ops.bonus_scan`` forms the decays and walks each
request's tokens from the state it left (float32 [heads, dim, dim] per request);
``ops.gated_norm`` norms every head's output, applies the weight and SiLU of the gate; the output
projection follows.  The state and everything inside the recurrence are 32-bit in both precisions.
"""
from __future__ import annotations

import torch

from ..cache.needs import FixedState
from ..config.spec import TensorSpec, TimeMixingSpec
from ..kernels import ops
from .base import Runtime, register_mixer

BLENDS = ("r", "k", "v", "g", "w")       # the order of the blended rows: four wide projections, then the decay's


@register_mixer("time_mixing")
class TimeMixing:
    can_defer_output = True
    graph_safe = True

    @staticmethod
    def tensor_specs(spec: TimeMixingSpec, prefix: str):
        inner = spec.heads * spec.dim
        return ([TensorSpec(f"{prefix}.mu.{name}", (spec.hidden,), "share") for name in BLENDS]
                + [TensorSpec(f"{prefix}.{name}", (inner, spec.hidden)) for name in BLENDS[:4]]
                + [TensorSpec(f"{prefix}.w1", (spec.rank, spec.hidden)),
                   TensorSpec(f"{prefix}.w2", (inner, spec.rank)),
                   TensorSpec(f"{prefix}.w0", (inner,), "log_rate"),
                   TensorSpec(f"{prefix}.u", (spec.heads, spec.dim), "share"),
                   TensorSpec(f"{prefix}.norm", (inner,), "norm"),
                   TensorSpec(f"{prefix}.o", (spec.hidden, inner))])

    def __init__(self, spec: TimeMixingSpec, tensors, runtime: Runtime):
        self.spec = spec
        self.mu = runtime.vector_f32(torch.stack([tensors[f"mu.{name}"] for name in BLENDS]))
        self.w_in = runtime.matrix(torch.stack([tensors[name] for name in BLENDS[:4]]))
        self.w1, self.w2 = runtime.matrix(tensors["w1"]), runtime.matrix(tensors["w2"])
        self.w_o = runtime.matrix(tensors["o"])
        self.w0, self.bonus = runtime.vector_f32(tensors["w0"]), runtime.vector_f32(tensors["u"].reshape(-1))
        self.norm_weight = runtime.vector_f32(tensors["norm"])
        self.act = runtime.precision.act
        self._state_dtype = runtime.precision.name

    def activation_elements(self) -> int:
        s = self.spec
        return len(BLENDS) * s.hidden + s.heads * s.dim * 14 + s.rank

    def cache_need(self):
        s = self.spec
        return (FixedState((s.heads, s.dim, s.dim), "float32", name="state"),
                FixedState((1, s.hidden), self._state_dtype, name="shift"))

    def heads_forward(self, x, ctx, cache, out, scale: float = 1.0) -> None:
        """Everything in front of the output projection, times ``scale``, into the rows ``out``."""
        s = self.spec
        if cache is None or not cache.writable:
            raise ValueError("a recurrent mixer needs a state of its own")
        rows = ops.token_blend(x, self.mu, cache.states["shift"], ctx)
        y = ops.linears_batched(rows[:, :4], self.w_in)
        a = ops.linear(ops.linear_act(rows[:, 4], self.w1, "tanh"), self.w2, out_dtype=torch.float32)
        o = ops.bonus_scan(y[:, 0], y[:, 1], y[:, 2], a, self.w0, self.bonus, cache.states["state"], ctx, s.heads, s.dim, s.dim)
        ops.gated_norm(o, self.norm_weight, y[:, 3], s.eps, s.heads, self.act, gate_function="silu", out=out, scale=scale)

    def forward(self, x, ctx, cache, defer_output: bool = False):
        out = torch.empty((x.shape[0], self.spec.heads * self.spec.dim), dtype=x.dtype, device=x.device)
        self.heads_forward(x, ctx, cache, out)
        if defer_output:
            return ops.linear_or_pending(out, self.w_o)
        return ops.linear(out, self.w_o)
