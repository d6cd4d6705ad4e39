"""Grouped-query attention with keys and values of different sizes, a norm of q and k (over the
whole projection, or head by head, with or without a weight), a sink term in the softmax, scores
with a query temperature, a soft cap and a learned bias over distances, an output gate per head or
per feature, values that may be the unnormed keys or a blend with an earlier layer's, projection
biases, and a causal, sliding-window or chunked mask (the formulas are with :class:`GatedAttentionSpec`).

One product makes [q | k | v | gate] (or [q | gate] for a layer that reads another layer's pages,
[q | k] for one whose values are its keys); ``ops.proj_norm_rope_cache`` or
``ops.head_norm_rope_cache`` norms q and k, rotates them and writes k and v into the pages; the
attention kernel applies the sink and the gate's sigmoid to every head's output; the output
projection follows.  In a step of single tokens the tensor-core decode kernels take the rows of
a layer with a norm per head raw and do the norm, the rotation and the page write themselves, as
they do for :class:`Attention`.  Biases and blended values enter in ``ops.head_norm_rope_cache`` or, where a
decode step has a handful of rows, in the product's epilogue; the first layer's values of a step travel
to the later ones through ``ctx.shared`` (a token's values are always of the same step).  Scores, softmax, the sink and the gate are 32-bit in both
precisions.  A chunked mask reaches the attention kernels as a negative window (minus the chunk's size).

A layer with a temperature, a soft cap, a distance bias or a gate per feature hands the attention
kernels a score form (``kernels.attention.score_form``): all of it happens inside them, the bias from a
table over distances that is laid out once from the checkpoint's buckets.  Those kernels also
take keys and values of different sizes.

Kernels: bfloat16 with key and value sizes that the tensor-core attention takes go through the
framework's paged kernels (tcgen05 prompt tiles, TMA decode; the sink enters their final
normalisation, the gate is one more kernel); every other shape, and the 32-bit path, runs
on CUDA cores in 32-bit arithmetic with sink and gate inside the kernel.
"""
from __future__ import annotations

import math
import os

import torch

from ..cache.needs import PagedKV
from ..config.spec import GatedAttentionSpec, TensorSpec
from ..kernels import ops
from ..kernels.attention import decode_fuses_input, paged_attention, score_form, supports_tensor_cores
from .base import POSITIONS, Runtime, register_mixer


# False (``MRUN_GATED_ATTENTION_TENSOR_CORES=0`` in the environment): the CUDA-core kernel for every
# shape (tests compare the two)
TENSOR_CORES = os.environ.get("MRUN_GATED_ATTENTION_TENSOR_CORES", "1") != "0"


def distance_buckets(rows: int, reach: float) -> list[int]:
    """The table row of every distance 0, 1, ... up to the first one that takes the last row (which
    every longer distance takes too)."""
    half, out = rows // 2, []
    for n in range(1 << 30):
        if n < half:
            b = n
        elif half < 1 or reach <= half:
            b = rows - 1
        else:
            b = min(rows - 1, half + math.floor(math.log(n / half) / math.log(reach / half) * (rows - half)))
        out.append(b)
        if b == rows - 1:
            return out


def half_split_order(dim: int, rotary_dim: int) -> list[int]:
    """The features of a head with its rotating pairs (2i, 2i + 1) moved to (i, i + rotary_dim / 2)."""
    return list(range(0, rotary_dim, 2)) + list(range(1, rotary_dim, 2)) + list(range(rotary_dim, dim))


@register_mixer("gated_attention")
class GatedAttention:
    accepts_normed_rows = True      # its first product takes ``ops.NormedRows`` as x
    can_defer_output = True

    @staticmethod
    def tensor_specs(spec: GatedAttentionSpec, prefix: str):
        nq, nk, nv = spec.heads * spec.dim, spec.kv_heads * spec.dim, spec.kv_heads * spec.vdim
        out = [TensorSpec(f"{prefix}.q", (nq, spec.hidden)),
               TensorSpec(f"{prefix}.o", (spec.hidden, spec.heads * spec.vdim))]
        if spec.own_kv:
            out.append(TensorSpec(f"{prefix}.k", (nk, spec.hidden)))
            if spec.values != "keys":
                out.append(TensorSpec(f"{prefix}.v", (nv, spec.hidden)))
        if spec.qk_norm not in (None, "unit"):
            per_head = spec.qk_norm == "head"
            out.append(TensorSpec(f"{prefix}.q.norm", (spec.dim if per_head else nq,), "norm"))
            if spec.own_kv:
                out.append(TensorSpec(f"{prefix}.k.norm", (spec.dim if per_head else nk,), "norm"))
        if spec.head_gate:
            out.append(TensorSpec(f"{prefix}.g", (spec.heads, spec.hidden)))
        if spec.element_gate:
            out.append(TensorSpec(f"{prefix}.g", (spec.heads * spec.vdim, spec.hidden)))
        if spec.distance_bias is not None:
            out.append(TensorSpec(f"{prefix}.rel", (spec.distance_bias[0], spec.heads), "normal"))
        if spec.biases:
            out += [TensorSpec(f"{prefix}.{name}.b", (n,)) for name, n in (("q", nq), ("k", nk), ("v", nv))]
        if spec.learned_sink:
            out.append(TensorSpec(f"{prefix}.sink", (spec.heads,)))
        if spec.value_mix is not None:
            out.append(TensorSpec(f"{prefix}.vmix", (), "share"))
        return out

    def __init__(self, spec: GatedAttentionSpec, tensors, runtime: Runtime):
        if spec.heads % spec.kv_heads:
            raise ValueError(f"heads={spec.heads} is not a multiple of kv_heads={spec.kv_heads}")
        if spec.qk_norm not in (None, "projection", "head", "unit"):
            raise ValueError(f"the q/k norm of this attention works over the whole projection or head by head, "
                             f"not {spec.qk_norm!r}")
        if spec.head_gate and spec.element_gate:
            raise ValueError("an attention has a gate per head or a gate per feature, not both")
        if spec.head_gate and (spec.soft_cap or spec.temperature or spec.distance_bias):
            raise ValueError("a gate per head does not go with scores that the kernels work on")
        if spec.soft_cap is not None and not spec.soft_cap > 0:
            raise ValueError(f"a soft cap must be positive, got {spec.soft_cap}")
        if spec.values not in ("projection", "keys"):
            raise ValueError(f"values come from a projection of their own or are the keys, not {spec.values!r}")
        self.keys_as_values = spec.values == "keys"
        if self.keys_as_values and (spec.vdim != spec.dim or not spec.own_kv):
            raise ValueError("values that are the keys have the keys' size and belong to a layer with keys of its own")
        if spec.window is not None and spec.chunk is not None:
            raise ValueError("an attention has a sliding window or a chunked mask, not both")
        if (spec.window is not None and spec.window < 1) or (spec.chunk is not None and spec.chunk < 1):
            raise ValueError("a window or a chunk holds at least one position")
        if spec.value_mix not in (None, "first", "blend"):
            raise ValueError(f"values are the first ones of the step or a blend with them, not {spec.value_mix!r}")
        if (spec.biases or spec.value_mix) and (spec.qk_norm == "projection" or not spec.own_kv or self.keys_as_values):
            raise ValueError("biases and mixed values go with keys and values of their own and without a norm over the projection")
        if spec.learned_sink and not spec.sink:
            raise ValueError("a learned sink is a sink")
        self.spec = spec
        self.runtime = runtime
        # what the attention kernels take as their window: W, 0 for none, -C for chunks of C
        self.mask = -spec.chunk if spec.chunk is not None else (spec.window or 0)
        self.nq, self.nk, self.nv = spec.heads * spec.dim, spec.kv_heads * spec.dim, spec.kv_heads * spec.vdim
        self.position = POSITIONS.build(spec.position, {}, runtime) if spec.position is not None else None
        self.pairing = getattr(self.position, "pairing", "half")
        biases = {name: tensors[f"{name}.b"] for name in "qkv"} if spec.biases else {}
        if self.pairing == "interleaved" and spec.qk_norm == "unit" and not self.keys_as_values:
            # the features of every q and k head in another order, pairs (2i, 2i + 1) as (i, i + n/2): scores and
            # a norm without a weight do not notice, and the kernels with half-split pairs take the layer
            tensors = dict(tensors)
            order = half_split_order(spec.dim, self.position.rotary_dim)
            for name in ("q", "k") if spec.own_kv else ("q",):
                tensors[name] = tensors[name].view(-1, spec.dim, spec.hidden)[:, order].reshape(tensors[name].shape)
                if spec.biases:
                    biases[name] = biases[name].view(-1, spec.dim)[:, order].reshape(-1)
            self.pairing = "half"
        parts = [tensors["q"]] + ([tensors["k"]] + ([] if self.keys_as_values else [tensors["v"]]) if spec.own_kv else [])
        self.k_off, self.v_off = (self.nq, -1 if self.keys_as_values else self.nq + self.nk) if spec.own_kv else (-1, -1)
        # the kernel that norms head by head also serves the layers that norm nothing special
        self.per_head = spec.qk_norm in ("head", "unit") or self.keys_as_values or spec.biases or spec.value_mix is not None
        self.gate_off = sum(p.shape[0] for p in parts)
        if spec.head_gate or spec.element_gate:
            parts.append(tensors["g"])
        rows = sum(p.shape[0] for p in parts)
        if rows % 8:        # rows of the product's output start on 16 bytes, as the tensor-core kernels read q
            parts.append(torch.zeros((8 - rows % 8, spec.hidden), dtype=parts[0].dtype, device=parts[0].device))
        self.w_in = runtime.matrix(torch.cat(parts, dim=0))
        self.b_in = self.b_rows = None          # biases of q, k and v; the same as long as the product's rows
        if spec.biases:
            b = torch.cat([biases[name].to(torch.float32) for name in "qkv"])
            self.b_in = runtime.vector_f32(b)
            self.b_rows = runtime.vector_f32(torch.cat([b, b.new_zeros(self.w_in.shape[0] - b.numel())]))
        self.v_share = float(tensors["vmix"]) if spec.value_mix == "blend" else 0.0
        self.sink = None
        if spec.sink:
            self.sink = (runtime.vector_f32(tensors["sink"]) if spec.learned_sink
                         else torch.zeros(spec.heads, dtype=torch.float32, device=runtime.device))
        self.w_o = runtime.matrix(tensors["o"])
        self.q_weight = self.k_weight = None
        if spec.qk_norm == "unit":          # a norm without a weight: a weight of ones
            self.q_weight = self.k_weight = torch.ones(spec.dim, dtype=torch.float32, device=runtime.device)
        elif spec.qk_norm is not None:
            self.q_weight = runtime.vector_f32(tensors["q.norm"])
            self.k_weight = runtime.vector_f32(tensors["k.norm"]) if spec.own_kv else None
        ratio = spec.heads // spec.kv_heads
        # scores or outputs that the attention kernels work on themselves
        self.formed = (spec.temperature is not None or spec.soft_cap is not None or spec.distance_bias is not None
                       or spec.element_gate)
        self.bias = None
        if spec.distance_bias is not None:
            at = torch.tensor(distance_buckets(*spec.distance_bias), dtype=torch.long)
            self.bias = runtime.vector_f32(tensors["rel"].to("cpu", torch.float32)[at].t())      # [heads, distances]
        # unit vectors times the root of their size: no product of two exceeds the size
        self.dot_bound = float(spec.dim) if spec.qk_norm == "unit" else math.inf
        self.tensor_cores = (TENSOR_CORES and supports_tensor_cores(runtime.precision.act, spec.dim, ratio, spec.vdim))
        # the tiled kernel that very wide groups fall to needs a tile list made on the host
        self.graph_safe = not (self.tensor_cores and ratio > 16)
        # rows laid out [q | k | v] with a norm per head and half-split pairs are what the decode
        # attention kernels take raw (they norm, rotate and store the step's q, k and v themselves)
        self.fusable = (self.tensor_cores and spec.qk_norm in ("head", "unit") and spec.own_kv and not self.keys_as_values
                        and self.pairing == "half")

    def cache_need(self):
        s = self.spec
        if not s.own_kv:
            return None
        # a chunk's keys lie within the last `chunk` positions: the pages before them are given back
        return PagedKV(s.kv_heads, s.dim, s.chunk if s.chunk is not None else s.window,
                       value_dim=s.vdim if s.vdim != s.dim else None)

    def activation_elements(self) -> int:
        s = self.spec
        kept = self.nv if s.value_mix is not None else 0
        return kept + 2 * self.nq + self.nk + self.nv + s.heads * (1 + 2 * s.vdim) + (s.heads * s.vdim if s.element_gate else 0)

    def heads_forward(self, x, ctx, cache, out, scale: float = 1.0) -> None:
        """Everything in front of the output projection: the gated heads into the rows ``out`` (which may
        be a column slice where the layer has a score form), times ``scale``."""
        s = self.spec
        if cache is None or cache.k is None:
            raise ValueError("this attention has no pages to read: a layer without keys and values of its own "
                             "runs as a schedule entry that names the cache of another")
        if s.own_kv != bool(cache.writable):
            raise ValueError("an attention with keys and values of its own writes its own pages, one without reads another's")
        group = ctx.group(cache.group_key)
        fuses = self.fusable and decode_fuses_input(ctx, x.dtype, s.heads, s.kv_heads, s.dim, self.runtime.page_size)
        plain = s.value_mix is None and not s.biases
        blend = (ctx.shared["first_values"], self.v_share) if s.value_mix == "blend" else None
        keep = None
        if fuses and not plain and ops.skinny_ok(x, self.w_in):
            # a handful of single tokens: biases and blended values come out of the product itself
            y = ops.linear_blended(x, self.w_in, self.b_rows, None if blend is None else (*blend, self.v_off))
            if s.value_mix == "first":
                ctx.shared["first_values"] = y[:, self.v_off:self.v_off + self.nv]
        else:
            fuses = fuses and plain
            y = ops.linear(x, self.w_in)
            if s.value_mix == "first":
                keep = ctx.shared["first_values"] = torch.empty((x.shape[0], self.nv), dtype=x.dtype, device=x.device)
        rot = self.position.rotation(ctx) if self.position is not None else None
        rotary_dim = self.position.rotary_dim if self.position is not None else 0
        gate = y[:, self.gate_off:self.gate_off + s.heads] if s.head_gate else None
        # a layer without a score form writes dense rows
        wanted, form = out, None
        if self.formed:
            form = score_form(out, s.soft_cap, s.temperature, self.bias,
                              y[:, self.gate_off:self.gate_off + s.heads * s.vdim] if s.element_gate else None, scale,
                              self.dot_bound)
        elif scale != 1.0 or not out.is_contiguous():
            out = torch.empty(out.shape, dtype=out.dtype, device=out.device)
        raw = None
        if fuses:
            # a pure decode step: the attention kernel norms, rotates and stores q, k, v itself
            raw = (self.q_weight, self.k_weight, s.eps, rot, rotary_dim, group.slot_mapping)
        elif self.per_head:
            ops.head_norm_rope_cache(y, 0, max(self.k_off, 0), self.v_off, s.heads, s.kv_heads, s.dim, s.vdim,
                                     self.q_weight, self.k_weight, s.eps, rot, rotary_dim, self.pairing,
                                     group.slot_mapping if s.own_kv else None, cache.k, cache.v, self.runtime.page_size,
                                     bias=self.b_in, keep=keep, blend=blend)
        else:
            ops.proj_norm_rope_cache(y, 0, self.k_off, self.v_off, s.heads, s.kv_heads, s.dim, s.vdim, self.q_weight,
                                     self.k_weight, s.eps, rot, rotary_dim, self.pairing,
                                     group.slot_mapping if s.own_kv else None, cache.k, cache.v, self.runtime.page_size)
        if self.tensor_cores:
            paged_attention(y, y.stride(0), out, cache, group, ctx, s.heads, s.softmax_scale, self.mask, raw=raw, sink=self.sink,
                            form=form)
            if gate is not None:
                ops.head_gate(out, gate, s.heads)
        else:
            ops.paged_attention_generic(y, y.stride(0), out, cache.k, cache.v, group.block_tables, ctx.token_slot,
                                        ctx.positions, s.heads, s.softmax_scale, self.mask, sink=self.sink, gate=gate, form=form)
        if out is not wanted:
            torch.mul(out, scale, out=wanted)

    def forward(self, x, ctx, cache, defer_output: bool = False):
        out = torch.empty((x.shape[0], self.spec.heads * self.spec.vdim), dtype=x.dtype, device=x.device)
        self.heads_forward(x, ctx, cache, out)
        if defer_output:
            return ops.linear_or_pending(out, self.w_o)
        return ops.linear(out, self.w_o)
