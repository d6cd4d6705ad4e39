"""Two mixers side by side (the formulas are with :class:`ParallelMixerSpec`).

Both read the same normed rows.  Each runs as it would alone, with its own kinds of cache: the
schedule entry's need is the two needs together (at most one of them paged; fixed-size states
under different names), and both see the entry's one :class:`EntryCache`, of which each uses its
own members.

``combine`` = ``"norm_mean"``: their last products write 32-bit sums; each branch is divided by its root mean
square over the model width, multiplied by its weight, and ``share`` of their sum joins the
stream.  A caller that takes pending outputs (``defer_output=True``) gets the two branches as
they are (``ops.PendingPairNorm``): a layer norm behind it does the branch norms, the average,
the residual sum and its own norm in one kernel; otherwise ``ops.pair_norm_mean`` makes the
32-bit addend.

``combine`` = ``"sum"``: where both sides offer ``heads_forward(x, ctx, cache, out, scale)`` (everything
in front of their output projection ``w_o``, times ``scale``), they fill the two halves of one
matrix of rows and one product with [W_o left | W_o right] makes the scaled sum; otherwise the two
outputs are added as they are.
"""
from __future__ import annotations

import torch

from ..cache.needs import split_need
from ..config.spec import ParallelMixerSpec, TensorSpec
from ..kernels import ops
from .base import MIXERS, Runtime, local, register_mixer


@register_mixer("parallel")
class ParallelMixer:
    can_defer_output = True         # ``forward(..., defer_output=True)`` may return ``ops.PendingPairNorm``

    @staticmethod
    def tensor_specs(spec: ParallelMixerSpec, prefix: str):
        out = []
        for side, name in ((spec.left, spec.left_prefix), (spec.right, spec.right_prefix)):
            out += MIXERS.tensor_specs(side, f"{prefix}.{name}")
            if spec.combine == "norm_mean":
                out.append(TensorSpec(f"{prefix}.{name}.{spec.out_name}", (spec.hidden,), "norm"))
        return out

    def __init__(self, spec: ParallelMixerSpec, tensors, runtime: Runtime):
        if spec.combine not in ("norm_mean", "sum"):
            raise ValueError(f"two mixers side by side are combined as norm_mean or sum, not {spec.combine!r}")
        self.spec = spec
        self.sides = []
        normed = spec.combine == "norm_mean"
        for side, name in ((spec.left, spec.left_prefix), (spec.right, spec.right_prefix)):
            mine = local(tensors, name)
            mixer = MIXERS.build(side, mine, runtime)
            self.sides.append((mixer, runtime.vector_f32(mine[spec.out_name]) if normed else None,
                               bool(getattr(mixer, "can_defer_output", False))))
        self.w_o = None         # the two output projections side by side; the sides' own are not used then
        if not normed and all(hasattr(mixer, "heads_forward") for mixer, _, _ in self.sides):
            self.w_o = torch.cat([mixer.w_o for mixer, _, _ in self.sides], dim=1).contiguous()
            self.widths = [mixer.w_o.shape[1] for mixer, _, _ in self.sides]
            for mixer, _, _ in self.sides:
                mixer.w_o = None
        split_need(self.cache_need())       # refuses two paged needs, and states of one name
        self.graph_safe = all(getattr(mixer, "graph_safe", False) for mixer, _, _ in self.sides)

    def cache_need(self):
        needs = []
        for mixer, _, _ in self.sides:
            need = mixer.cache_need()
            if need is not None:
                needs += list(need) if isinstance(need, (tuple, list)) else [need]
        return tuple(needs) if needs else None

    def activation_elements(self) -> int:
        total = 2 * self.spec.hidden if self.w_o is None else self.w_o.shape[1]
        for mixer, _, _ in self.sides:
            hint = getattr(mixer, "activation_elements", None)
            total += int(hint()) if hint is not None else 0
        return total

    def _branch(self, mixer, defers: bool, x, ctx, cache) -> torch.Tensor:
        """One side's output as 32-bit rows."""
        if defers:
            y = mixer.forward(x, ctx, cache, defer_output=True)
            if isinstance(y, ops.PendingLinear):
                return y.compute(torch.float32)
        else:
            y = mixer.forward(x, ctx, cache)
        if isinstance(y, ops.PENDING):
            y = y.compute()
        return y if y.dtype == torch.float32 else y.to(torch.float32)

    def forward(self, x, ctx, cache, defer_output: bool = False):
        (left, w_left, left_defers), (right, w_right, right_defers) = self.sides
        if self.w_o is not None:
            width = self.w_o.shape[1]           # rows start on 16 bytes
            rows = torch.empty((x.shape[0], -(-width // 8) * 8), dtype=x.dtype, device=x.device)[:, :width]
            left.heads_forward(x, ctx, cache, rows[:, :self.widths[0]], self.spec.scales[0])
            right.heads_forward(x, ctx, cache, rows[:, self.widths[0]:], self.spec.scales[1])
            return ops.linear_or_pending(rows, self.w_o) if defer_output else ops.linear(rows, self.w_o)
        a = self._branch(left, left_defers, x, ctx, cache)
        b = self._branch(right, right_defers, x, ctx, cache)
        if self.spec.combine == "sum":
            return ops.scale(a, self.spec.scales[0]).add_(ops.scale(b, self.spec.scales[1]))
        pending = ops.PendingPairNorm(a, b, w_left, w_right, self.spec.eps, self.spec.share)
        return pending if defer_output else pending.compute()
