"""Latent attention over a paged cache of one latent row per token.

The cache row of a token is ``[c | r | 0...]``: its key/value latent c (``kv_rank`` features,
RMS-normed), the rotated key part r that all heads share (``rot_dim`` features) and zeros up to a
width the attention kernels take.  Keys and values of the heads are never made: with
K_h = U_h c and V_h = W_h c (the two up-projections), a head's score is

    q_plain . (U_h c) + q_rot . r  =  (U_h^T q_plain) . c + q_rot . r,

so the query row ``[U_h^T q_plain | q_rot | 0...]`` meets the cache row as one key of a single
key/value head, and the head's output is W_h (sum_j p_j c_j): the same cache row is the value,
and W_h runs on the weighted latent.  The framework's paged attention kernels therefore serve
this mixer unchanged (``heads`` query heads over one kv head whose K and V are the same pages);
prefill, decode and mixed steps take the paths they take for grouped-query attention.  Rows wider
than those kernels' 256 features (a latent of 512, say) go to a tensor-core kernel of their own
(``csrc/attention_latent.cu``: a block a token and 16 heads, a quarter of the value columns a warp), and
so do steps of single tokens with more than 16 heads (without a window).

A layer without a query latent (``q_rank`` = 0) has one query projection ``q`` straight from the
input; it rides in the same product as the key/value down-projection, and so do the rows of a gate
per head, whose sigmoid multiplies the heads behind W_h.  A layer without positions (``rot_dim`` = 0)
caches the latent alone.  ``window`` reaches the
attention kernels as it does for grouped-query attention.

**Steps with prompt portions** of a layer without positions and without a window, where the heads' plain keys
and values are 64 or 128 features, make the keys and values after all (``_expanded``): the scores of a
portion against its own context cost (dim + vdim) a key and head that way against 2 kv_rank, and the tcgen05
kernel takes the shape.  The contexts' latents are gathered out of the pages, each segment's keys and
values become one large page of scratch, and the paged kernels run over those.  Only while the contexts
together are not much longer than the step (``EXPAND_ROWS`` times its rows), so that a long context is not
projected up again for every portion of it; other steps, decode steps and the 32-bit path stay with the
latent.

Per step: one product for both down-projections (their weights stacked), one kernel that norms
the two latents, rotates r and writes the cache row, the query up-projection, a per-head product
with U_h^T, one kernel that rotates the queries' rotated parts into the query rows, attention, a
per-head product with W_h, the output projection (left pending for the norm after it).
"""
from __future__ import annotations

import numpy as np
import torch

from ..cache.needs import PagedLatent
from ..config.spec import LatentAttentionSpec, TensorSpec
from ..kernels import ops
from ..kernels.attention import latent_wide_ok, paged_attention, supports_tensor_cores
from .base import POSITIONS, Runtime, register_mixer


EXPAND_ROWS = 4             # rows of scratch a step's row may bring with it where keys and values are made
EXPAND_SEGMENTS = 8         # and the most segments (each is two products of its own)


class _Pages:
    """Scratch keys and values as the attention kernels take a cache: a page a segment."""

    def __init__(self, k, v, table):
        self.k, self.v, self.block_tables, self.max_blocks = k, v, table, 1


@register_mixer("latent_attention")
class LatentAttention:
    accepts_normed_rows = True      # its first product takes ``ops.NormedRows`` as x
    can_defer_output = True         # ``forward(..., defer_output=True)`` may return ``ops.PendingLinear``

    @staticmethod
    def tensor_specs(spec: LatentAttentionSpec, prefix: str):
        s = spec
        if s.q_rank:
            query = [TensorSpec(f"{prefix}.dq", (s.q_rank, s.hidden)),
                     TensorSpec(f"{prefix}.dq.norm", (s.q_rank,), "norm"),
                     TensorSpec(f"{prefix}.uq", (s.heads * (s.dim + s.rot_dim), s.q_rank))]
        else:
            query = [TensorSpec(f"{prefix}.q", (s.heads * (s.dim + s.rot_dim), s.hidden))]
        gate = [TensorSpec(f"{prefix}.g", (s.heads, s.hidden))] if s.head_gate else []
        return query + gate + [
            TensorSpec(f"{prefix}.dkv", (s.kv_rank + s.rot_dim, s.hidden)),
            TensorSpec(f"{prefix}.dkv.norm", (s.kv_rank,), "norm"),
            TensorSpec(f"{prefix}.uk", (s.heads * s.dim, s.kv_rank)),
            TensorSpec(f"{prefix}.uv", (s.heads * s.vdim, s.kv_rank)),
            TensorSpec(f"{prefix}.o", (s.hidden, s.heads * s.vdim)),
        ]

    def __init__(self, spec: LatentAttentionSpec, tensors, runtime: Runtime):
        s = self.spec = spec
        self.runtime = runtime
        if s.window is not None and s.window < 1:
            raise ValueError("a window holds at least one position")
        # the first product: [query latent | key/value latent | shared key part], or, without a
        # query latent, [queries | key/value latent | shared key part]
        parts = [tensors["dq" if s.q_rank else "q"], tensors["dkv"]]
        self.gate_off = sum(p.shape[0] for p in parts)
        if s.head_gate:
            parts.append(tensors["g"])
        if not s.q_rank:        # zero rows at the end: the queries in the product's rows start on 16 bytes
            rows = sum(p.shape[0] for p in parts)
            parts.append(torch.zeros((-rows % 8, s.hidden), dtype=parts[0].dtype, device=parts[0].device))
        self.w_down = runtime.matrix(torch.cat(parts, dim=0))
        self.q_norm = runtime.vector_f32(tensors["dq.norm"]) if s.q_rank else None
        self.kv_norm = runtime.vector_f32(tensors["dkv.norm"])
        self.w_uq = runtime.matrix(tensors["uq"]) if s.q_rank else None
        # U_h^T per head, [heads, kv_rank, dim]: the per-head product takes weights as [out, in]
        self.w_uk_t = runtime.matrix(tensors["uk"].view(s.heads, s.dim, s.kv_rank).transpose(1, 2))
        self.w_uv = runtime.matrix(tensors["uv"].view(s.heads, s.vdim, s.kv_rank))
        self.w_o = runtime.matrix(tensors["o"])
        self.position = POSITIONS.build(s.position, {}, runtime) if s.position is not None else None
        self.rot_dims = self.position.rotary_dim if self.position is not None else 0
        self.pairing = getattr(self.position, "pairing", "half")
        if self.rot_dims > s.rot_dim:
            raise ValueError(f"{self.rot_dims} rotating features do not fit the rotated part of {s.rot_dim}")
        # the cache row's width: a size the tensor-core attention kernels are built for
        self.width = -(-(s.kv_rank + s.rot_dim) // 16) * 16
        # the tiled kernel that very wide groups fall to needs a tile list made on the host; without a
        # window the single tokens of such groups have the kernel for wide rows
        self.graph_safe = not (supports_tensor_cores(runtime.precision.act, self.width, s.heads) and s.heads > 16
                               and (s.window is not None or not latent_wide_ok(runtime.precision.act, self.width, s.kv_rank)))

        self.expandable = (runtime.precision.act == torch.bfloat16 and s.rot_dim == 0 and not s.q_rank and s.window is None
                           and s.dim in (64, 128) and s.vdim in (64, 128))

    def _scratch_rows(self, ctx) -> int:
        """Rows of the scratch pages of a step whose keys and values are made, 0 for a step that keeps the latent."""
        if not self.expandable or ctx.max_q_len == 1 or len(ctx.segments) > EXPAND_SEGMENTS:
            return 0
        rows = 128
        while rows < ctx.max_kv_len:
            rows *= 2
        return rows if rows * len(ctx.segments) <= EXPAND_ROWS * max(128, ctx.num_tokens) else 0

    def _expanded(self, q, ctx, cache, group, rows: int) -> torch.Tensor:
        """The heads' outputs over keys and values made from the contexts' latents: [tokens, heads * vdim]."""
        s, n = self.spec, len(ctx.segments)
        latents = ops.latent_rows(cache.k, group.block_tables, ctx.seg_slot[:n], ctx.seg_kv_len[:n], rows, s.kv_rank)
        k = torch.empty((n, s.heads, rows, s.dim), dtype=q.dtype, device=q.device)
        v = torch.empty((n, s.heads, rows, s.vdim), dtype=q.dtype, device=q.device)
        for i, seg in enumerate(ctx.segments):
            used = -(-(seg.pos_start + seg.q_len) // 128) * 128
            c = latents[i, :used].expand(s.heads, used, s.kv_rank)
            torch.bmm(c, self.w_uk_t, out=k[i, :, :used])
            torch.bmm(c, self.w_uv.transpose(1, 2), out=v[i, :, :used])
        table = ctx.shared.get("segment_pages")
        if table is None:           # state slot -> its segment's page
            pages = np.full(group.block_tables.shape[0], -1, dtype=np.int32)
            pages[[seg.slot for seg in ctx.segments]] = np.arange(n, dtype=np.int32)
            table = ctx.shared["segment_pages"] = ctx.upload(pages).view(-1, 1)
        scratch = _Pages(k, v, table)
        out = torch.empty((q.shape[0], s.heads * s.vdim), dtype=q.dtype, device=q.device)
        return paged_attention(q, q.stride(0), out, scratch, scratch, ctx, s.heads, s.softmax_scale, 0)

    def cache_need(self):
        return PagedLatent(self.width, self.spec.window)

    def activation_elements(self) -> int:
        s = self.spec
        latent = s.q_rank + s.kv_rank + s.rot_dim + s.heads * (s.dim + s.rot_dim + 2 * self.width + s.vdim)
        return latent + (EXPAND_ROWS * (s.kv_rank + s.heads * (s.dim + s.vdim)) if self.expandable else 0)

    def forward(self, x, ctx, cache, defer_output: bool = False):
        s, width = self.spec, self.width
        tokens = x.shape[0]
        group = ctx.group(cache.group_key)
        down = ops.linear(x, self.w_down)
        gate = down[:, self.gate_off:self.gate_off + s.heads] if s.head_gate else None
        down = down[:, :self.gate_off]
        rot = self.position.rotation(ctx) if self.position is not None else None
        slots = group.slot_mapping if cache.writable else None
        if s.q_rank:
            cq = torch.empty((tokens, s.q_rank), dtype=x.dtype, device=x.device)
            ops.latent_prepare(down, self.q_norm, self.kv_norm, s.eps, rot, self.rot_dims, self.pairing, slots, cq,
                               cache.k, s.q_rank, s.kv_rank, s.rot_dim)
            q = ops.linear(cq, self.w_uq)
        else:
            nq = s.heads * (s.dim + s.rot_dim)
            q = down[:, :nq]
            ops.latent_prepare(down[:, nq:], None, self.kv_norm, s.eps, rot, self.rot_dims, self.pairing, slots, None,
                               cache.k, 0, s.kv_rank, s.rot_dim)
        rows = self._scratch_rows(ctx)
        if rows and cache.writable:
            value = self._expanded(q, ctx, cache, group, rows)
            if gate is not None:
                ops.head_gate(value, gate, s.heads)
            return ops.linear_or_pending(value, self.w_o) if defer_output else ops.linear(value, self.w_o)
        q_att = torch.empty((tokens, s.heads, width), dtype=x.dtype, device=x.device)
        ops.linears_batched(q.unflatten(1, (s.heads, s.dim + s.rot_dim))[:, :, :s.dim], self.w_uk_t,
                            out=q_att[:, :, :s.kv_rank])
        if width > s.kv_rank:       # a rotated part, or zeros up to the row's width
            ops.latent_query(q, rot, self.rot_dims, self.pairing, q_att, s.heads, s.dim, s.rot_dim, s.kv_rank)
        mixed = torch.empty((tokens, s.heads * width), dtype=x.dtype, device=x.device)
        paged_attention(q_att.view(tokens, s.heads * width), s.heads * width, mixed, cache, group, ctx, s.heads,
                        s.softmax_scale, s.window or 0, value_dim=s.kv_rank)
        value = torch.empty((tokens, s.heads, s.vdim), dtype=x.dtype, device=x.device)
        ops.linears_batched(mixed.view(tokens, s.heads, width)[:, :, :s.kv_rank], self.w_uv, gate=gate, out=value)
        value = value.view(tokens, s.heads * s.vdim)
        if defer_output:
            return ops.linear_or_pending(value, self.w_o)
        return ops.linear(value, self.w_o)
