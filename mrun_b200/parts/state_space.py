"""Selective state-space mixer with a scalar decay per head (the formulas are with
:class:`StateSpaceSpec`).

One product makes [z | x | B | C | dt]; ``ops.causal_conv`` runs the short convolution with its bias and
SiLU over the contiguous [x | B | C] columns, from and into the request's last inputs;
``ops.ssm_scan`` forms steps and decays and walks each request's tokens from the state it left
(float32 [heads, state, vdim] per request); ``ops.skip_gate_norm`` adds the skip D x, applies SiLU of z
and then the norm of every part and its weight; the output projection follows.  The state and
everything inside the recurrence are 32-bit in both precisions.
"""
from __future__ import annotations

import torch

from ..cache.needs import FixedState
from ..config.spec import StateSpaceSpec, TensorSpec
from ..kernels import ops
from .base import Runtime, register_mixer


@register_mixer("state_space")
class StateSpace:
    can_defer_output = True
    graph_safe = True

    @staticmethod
    def tensor_specs(spec: StateSpaceSpec, prefix: str):
        inner = spec.heads * spec.vdim
        channels = inner + 2 * spec.groups * spec.state
        return [TensorSpec(f"{prefix}.in", (inner + channels + spec.heads, spec.hidden)),
                TensorSpec(f"{prefix}.conv", (channels, spec.conv), "taps"),
                TensorSpec(f"{prefix}.conv.b", (channels,)),
                TensorSpec(f"{prefix}.dt_bias", (spec.heads,), "log_rate"),
                TensorSpec(f"{prefix}.A_log", (spec.heads,), "log_rate"),
                TensorSpec(f"{prefix}.D", (spec.heads,), "norm"),
                TensorSpec(f"{prefix}.norm", (inner,), "norm"),
                TensorSpec(f"{prefix}.o", (spec.hidden, inner))]

    def __init__(self, spec: StateSpaceSpec, tensors, runtime: Runtime):
        if spec.heads % spec.groups:
            raise ValueError(f"heads={spec.heads} is not a multiple of groups={spec.groups}")
        self.spec = spec
        self.inner = spec.heads * spec.vdim
        if self.inner % spec.norm_groups:
            raise ValueError(f"{spec.norm_groups} norm groups do not divide {self.inner} features")
        self.channels = self.inner + 2 * spec.groups * spec.state
        w_in = tensors["in"]
        rows = w_in.shape[0]
        if rows % 8:        # rows of the product's output start on 16 bytes
            w_in = torch.cat([w_in, torch.zeros((8 - rows % 8, spec.hidden), dtype=w_in.dtype, device=w_in.device)], dim=0)
        self.w_in, self.w_o = runtime.matrix(w_in), runtime.matrix(tensors["o"])
        self.conv_weight, self.conv_bias = runtime.vector_f32(tensors["conv"]), runtime.vector_f32(tensors["conv.b"])
        self.dt_bias, self.a_log = runtime.vector_f32(tensors["dt_bias"]), runtime.vector_f32(tensors["A_log"])
        self.skip, self.norm_weight = runtime.vector_f32(tensors["D"]), runtime.vector_f32(tensors["norm"])
        self._state_dtype = runtime.precision.name

    def activation_elements(self) -> int:
        s = self.spec
        return 6 * self.inner + 2 * self.channels + 4 * s.groups * s.state + 3 * s.heads

    def cache_need(self):
        s = self.spec
        return (FixedState((s.heads, s.state, s.vdim), "float32", name="state"),
                FixedState((s.conv - 1, self.channels), self._state_dtype, name="conv"))

    def forward(self, x, ctx, cache, defer_output: bool = False):
        s = self.spec
        if cache is None or not cache.writable:
            raise ValueError("a recurrent mixer needs a state of its own")
        inner, keyed = self.inner, s.groups * s.state
        y = ops.linear(x, self.w_in)
        dt = y[:, inner + self.channels:inner + self.channels + s.heads]
        xbc = ops.causal_conv(y[:, inner:inner + self.channels], self.conv_weight, cache.states["conv"], ctx, residual=False,
                              silu=True, bias=self.conv_bias)
        o = ops.ssm_scan(xbc[:, inner + keyed:], xbc[:, inner:inner + keyed], xbc[:, :inner], dt, self.dt_bias, self.a_log,
                         cache.states["state"], ctx, s.heads, s.groups, s.state, s.vdim)
        o = ops.skip_gate_norm(o, xbc[:, :inner], self.skip, y[:, :inner], self.norm_weight, s.eps, s.norm_groups)
        if defer_output:
            return ops.linear_or_pending(o, self.w_o)
        return ops.linear(o, self.w_o)
