"""Selective state-space mixer with a decay per channel and state (the formulas are with
:class:`SelectiveScanSpec`).

One product makes [x | z]; ``ops.causal_conv`` runs the short convolution with its bias and SiLU over x, from and
into the request's last inputs; one product of x makes [r | B | C] (two where the step has more than single
tokens, so that B and C come in 32-bit), one of r the raw steps (32-bit output, as they enter the recurrence); ``ops.selective_scan`` forms steps and decays, walks each request's tokens
from the state it left (float32 [inner, state] per request) and applies the skip and the gate; the output
projection follows.  r is padded with zero columns up to a size the decode GEMM takes.  The state and
everything inside the recurrence are 32-bit in both precisions.
"""
from __future__ import annotations

import torch

from ..cache.needs import FixedState
from ..config.spec import SelectiveScanSpec, TensorSpec
from ..kernels import ops
from .base import Runtime, register_mixer


def _padded_rows(w: torch.Tensor, unit: int) -> torch.Tensor:
    extra = -w.shape[0] % unit
    return torch.cat([w, w.new_zeros((extra, *w.shape[1:]))], dim=0) if extra else w


@register_mixer("selective_scan")
class SelectiveScan:
    accepts_normed_rows = True      # its first product takes ``ops.NormedRows`` as x
    can_defer_output = True
    graph_safe = True

    @staticmethod
    def tensor_specs(spec: SelectiveScanSpec, prefix: str):
        return [TensorSpec(f"{prefix}.in", (2 * spec.inner, spec.hidden)),
                TensorSpec(f"{prefix}.conv", (spec.inner, spec.conv), "taps"),
                TensorSpec(f"{prefix}.conv.b", (spec.inner,)),
                TensorSpec(f"{prefix}.x", (spec.dt_rank + 2 * spec.state, spec.inner)),
                TensorSpec(f"{prefix}.dt", (spec.inner, spec.dt_rank)),
                TensorSpec(f"{prefix}.dt.b", (spec.inner,), "log_rate"),
                TensorSpec(f"{prefix}.A_log", (spec.inner, spec.state), "log_rate"),
                TensorSpec(f"{prefix}.D", (spec.inner,), "norm"),
                TensorSpec(f"{prefix}.o", (spec.hidden, spec.inner))]

    def __init__(self, spec: SelectiveScanSpec, tensors, runtime: Runtime):
        self.spec = spec
        w_x = tensors["x"]
        # [r | zeros | B | C | zeros]: r as wide as the decode GEMM's steps, rows on 16 bytes
        self.rank = -(-spec.dt_rank // 32) * 32
        r, bc = w_x[:spec.dt_rank], w_x[spec.dt_rank:]
        self.w_in = runtime.matrix(_padded_rows(tensors["in"], 8))
        self.w_x = runtime.matrix(_padded_rows(torch.cat([_padded_rows(r, 32), bc], dim=0), 8))
        self.w_dt = runtime.matrix(_padded_rows(tensors["dt"].t(), 32).t())
        self.w_o = runtime.matrix(tensors["o"])
        self.conv_weight, self.conv_bias = runtime.vector_f32(tensors["conv"]), runtime.vector_f32(tensors["conv.b"])
        self.dt_bias, self.skip = runtime.vector_f32(tensors["dt.b"]), runtime.vector_f32(tensors["D"])
        self.rates = runtime.vector_f32(-torch.exp(tensors["A_log"].to(torch.float64)))
        self._state_dtype = runtime.precision.name

    def activation_elements(self) -> int:
        s = self.spec
        # the raw steps are 32-bit: two elements each where the activations are 16-bit
        return 6 * s.inner + self.rank + 2 * s.state

    def cache_need(self):
        s = self.spec
        return (FixedState((s.inner, s.state), "float32", name="state"),
                FixedState((s.conv - 1, s.inner), self._state_dtype, name="conv"))

    def forward(self, x, ctx, cache, defer_output: bool = False):
        s = self.spec
        if cache is None or not cache.writable:
            raise ValueError("a recurrent mixer needs a state of its own")
        xz = ops.linear(x, self.w_in)
        u = ops.causal_conv(xz[:, :s.inner], self.conv_weight, cache.states["conv"], ctx, residual=False, silu=True,
                            bias=self.conv_bias)
        if ctx.max_q_len == 1:
            rbc = ops.linear(u, self.w_x)
            r, bc = rbc[:, :self.rank], rbc[:, self.rank:]
        else:
            r, bc = ops.linear(u, self.w_x[:self.rank]), ops.linear(u, self.w_x[self.rank:], out_dtype=torch.float32)
        dt = ops.linear(r, self.w_dt, out_dtype=torch.float32)
        o = ops.selective_scan(u, xz[:, s.inner:2 * s.inner], dt, self.dt_bias, self.rates, bc[:, :s.state],
                               bc[:, s.state:2 * s.state], self.skip, cache.states["state"], ctx)
        if defer_output:
            return ops.linear_or_pending(o, self.w_o)
        return ops.linear(o, self.w_o)
