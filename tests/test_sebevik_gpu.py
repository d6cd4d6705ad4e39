"""Sebevik on the GPU against the plain implementation (``plain_sebevik``): every new kernel and every part alone
(whole requests, token by token, portions down to one and two tokens, unequal requests side by side,
state slots and pages given back and used again), inputs made so that one far key, a window's edge, a
learned sink, an earlier layer's values or a kept state decides the result, then whole models replayed
through ``bin/trace_run`` cut in every way, then greedy generation through ``Engine.generate`` and the
command line."""
from __future__ import annotations

import numpy as np
import pytest
import torch

import plain_sebevik as plain
from test_fikudra_gpu import (LENGTHS, SIZES, TRACE_LENGTHS, Steps, check_rows, close, close_calls, named, random_tensors,
                              runtime)
from test_nisotar_gpu import edge_cuts, run_cut
from tiny_sebevik import STINY, attention, latent, lively, load_folder, mamba1, make_folder, moe, sconfig, tokens_of
from trace_tools import TraceBuilder, TraceRunner, cut_decode_tail, cut_mixed, cut_portions, cut_whole

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64


def tight(dtype):
    return 1e-5 if dtype == "float32" else 1e-2


# ------------------------------------------------------------------ kernels alone

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("hidden", [8, 100, 1027, 4096, 13000])
def test_norm_with_a_second_branch(dtype, hidden):
    """The residual sum takes a branch in 32-bit or in the activation type and a second one with a factor a
    row (zero for some rows); in place and at chosen rows."""
    from mrun_b200.kernels import ops
    act = getattr(torch, dtype)
    gen = torch.Generator().manual_seed(hidden)
    rand = lambda *s: torch.randn(*s, generator=gen)
    resid, delta, extra = rand(7, hidden) * 2, rand(7, hidden), rand(7, hidden).to(act)
    share, w = torch.tensor([0.5, 0.0, -1.5, 0.25, 0.0, 2.0, 1.0]), 1 + 0.3 * rand(hidden)
    rows = torch.tensor([6, 1, 2], dtype=torch.int32)
    for d in (None, delta, delta.to(act)):
        for scaled in (None, (extra.to(DEV), share.to(DEV))):
            total = resid.double() + (0 if d is None else d.double())
            if scaled is not None:
                total = total + share.double()[:, None] * extra.double()
            want = plain.unit_rms(total, 1e-5) * w.double()
            stream, out = resid.to(DEV), torch.empty((7, hidden), dtype=act, device=DEV)
            dd = None if d is None else d.to(DEV)
            ops.add_rmsnorm(stream, dd, w.to(DEV), 1e-5, out, scaled=scaled)
            close(out, want, dtype, "all rows", bound=tight(dtype))
            close(stream, total, "float32", "the stream", bound=1e-6)
            stream, out = resid.to(DEV), torch.empty((3, hidden), dtype=act, device=DEV)
            ops.add_rmsnorm(stream, dd, w.to(DEV), 1e-5, out, rows=rows.to(DEV), scaled=scaled)
            close(out, want[rows.long()], dtype, "chosen rows", bound=tight(dtype))
            assert torch.equal(stream.cpu(), resid)
    y = delta.to(act).to(DEV)
    ops.add_scaled_rows(y, extra.to(DEV), share.to(DEV))
    close(y, delta.to(act).double() + share.double()[:, None] * extra.double(), dtype, "scaled rows", bound=tight(dtype))
    y = delta.to(DEV)
    ops.add_scaled_rows(y, extra.to(DEV), share.to(DEV))
    close(y, delta.double() + share.double()[:, None] * extra.double(), "float32", "scaled rows onto 32-bit", bound=1e-6)


@pytest.mark.parametrize("rows, k, n", [(1, 64, 96), (5, 96, 160), (11, 1024, 64), (16, 64, 2048), (40, 96, 64)])
def test_pending_product_with_scaled_rows(rows, k, n):
    """A product left pending with rows that join it: folded into the decode GEMM's residual epilogue, added
    in the norm's pass behind the vendor product, or computed; the same sum each way."""
    from mrun_b200.config.spec import RMSNormSpec
    from mrun_b200.kernels import ops
    from mrun_b200.parts import NORMS
    gen = torch.Generator().manual_seed(rows * n)
    x = torch.randn(rows, k, generator=gen).to(torch.bfloat16)
    w = (torch.randn(n, k, generator=gen) * k ** -0.5).to(torch.bfloat16)
    extra = torch.randn(rows, n, generator=gen).to(torch.bfloat16)
    share = torch.rand(rows, generator=gen) * (torch.arange(rows) % 3 > 0)
    resid, weight = torch.randn(rows, n, generator=gen), 1 + 0.2 * torch.randn(n, generator=gen)
    branch = x.double() @ w.double().T + share.double()[:, None] * extra.double()
    total = resid.double() + branch
    norm = NORMS.build(RMSNormSpec(n, 1e-5, bare=True), {"": weight}, runtime("bfloat16"))
    pending = ops.PendingLinear(x.to(DEV), w.to(DEV), (extra.to(DEV), share.to(DEV)))
    close(pending.compute(), branch, "bfloat16", "computed", bound=1e-2)
    close(pending.compute(torch.float32), branch, "float32", "computed in 32-bit", bound=1e-5)
    stream = resid.to(DEV)
    h = norm.add_forward(stream, pending)
    if rows <= 16:
        assert isinstance(h, ops.NormedRows)
        h = h.finish()
    close(stream, total, "float32", "the stream", bound=1e-5)
    close(h, plain.unit_rms(total, 1e-5) * weight.double(), "bfloat16", "the normed rows", bound=2e-2)
    stream = resid.to(DEV)
    at = torch.tensor([rows - 1, 0], dtype=torch.int32, device=DEV)
    close(norm.rows_forward(stream, pending, at), (plain.unit_rms(total, 1e-5) * weight.double())[[rows - 1, 0]], "bfloat16",
          "chosen rows", bound=2e-2)
    assert torch.equal(stream.cpu(), resid)


@pytest.mark.parametrize("rows, n, k", [(1, 40, 32), (9, 200, 64), (16, 4096, 96), (3, 24, 2048)])
def test_product_with_a_bias_and_blended_columns(rows, n, k):
    from mrun_b200.kernels import ops
    gen = torch.Generator().manual_seed(n)
    x = torch.randn(rows, k, generator=gen).to(torch.bfloat16)
    w = (torch.randn(n, k, generator=gen) * k ** -0.5).to(torch.bfloat16)
    b = torch.randn(n, generator=gen)
    first = torch.randn(rows, 3 * n, generator=gen).to(torch.bfloat16)[:, n // 2:n // 2 + 8 * (n // 16)]
    column, share = n - first.shape[1] - 3, 0.3
    want = x.double() @ w.double().T + b.double()
    close(ops.linear_blended(x.to(DEV), w.to(DEV), b.to(DEV)), want, "bfloat16", "bias", bound=1e-2)
    at = slice(column, column + first.shape[1])
    want[:, at] = (1 - share) * want[:, at] + share * first.double()
    got = ops.linear_blended(x.to(DEV), w.to(DEV), b.to(DEV), (first.to(DEV), share, column))
    close(got, want, "bfloat16", "blend", bound=1e-2)
    got = ops.linear_blended(x.to(DEV), w.to(DEV), b.to(DEV), (first.to(DEV), share, column), "relu2")
    close(got, torch.relu(want) ** 2, "bfloat16", "activation", bound=2e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows, batch, n, k", [(1, 4, 64, 64), (16, 3, 40, 96), (5, 2, 24, 37), (40, 4, 64, 96)])
def test_batched_products_with_gates_into_strided_rows(dtype, rows, batch, n, k):
    from mrun_b200.kernels import ops
    act = getattr(torch, dtype)
    gen = torch.Generator().manual_seed(rows * n + k)
    x = torch.randn(rows, batch, k, generator=gen).to(act)
    w = (torch.randn(batch, n, k, generator=gen) * k ** -0.5).to(act)
    gate = torch.randn(rows, batch + 5, generator=gen).to(act)
    want = torch.einsum("tbk,bnk->tbn", x.double(), w.double())
    wide = torch.full((rows, batch, n + 8), 7.0, dtype=act, device=DEV)
    ops.linears_batched(x.to(DEV), w.to(DEV), out=wide[:, :, :n])
    close(wide[:, :, :n], want, dtype, "into strided rows", bound=tight(dtype))
    assert bool((wide[:, :, n:] == 7.0).all())
    got = ops.linears_batched(x.to(DEV), w.to(DEV), gate=gate.to(DEV)[:, 3:3 + batch])
    close(got, want * torch.sigmoid(gate[:, 3:3 + batch].double())[:, :, None], dtype, "gated", bound=2 * tight(dtype))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads, kv_heads, dim, vdim, rot_dims", [(4, 2, 64, 64, 32), (3, 1, 20, 28, 8), (2, 2, 128, 64, 128), (5, 5, 16, 40, 0),
                                                                  (4, 1, 80, 48, 80)])
def test_norm_rotation_and_pages_with_biases_and_values(dtype, heads, kv_heads, dim, vdim, rot_dims):
    """Biases before the norm, values kept (also for rows without a page) and blended, on both forms of the
    kernel."""
    from mrun_b200.kernels import ops
    act = getattr(torch, dtype)
    gen = torch.Generator().manual_seed(dim + vdim)
    tokens, page, share = 9, 4, 0.35
    nq, nk, nv = heads * dim, kv_heads * dim, kv_heads * vdim
    x = torch.randn(tokens, nq + nk + nv + 8, generator=gen).to(act)
    bias = torch.randn(nq + nk + nv, generator=gen)
    first = torch.randn(tokens, nv + 16, generator=gen).to(act)[:, 8:8 + nv]
    slots = torch.tensor([9, 2, 40, -1, 17, 5, 0, 31, 30], dtype=torch.int32)
    rot = None
    if rot_dims:
        angle = (torch.arange(tokens) * 3).double()[:, None] * 100.0 ** (-2.0 * torch.arange(rot_dims // 2, dtype=F64) / rot_dims)
        rot = torch.stack([torch.cos(angle), torch.sin(angle)], dim=-1).float()
    biased = x[:, :nq + nk + nv].double() + bias.double()

    def turned(v):
        y = plain.unit_rms(v, 1e-5)
        if rot is not None:
            c, s = rot[:, None, :, 0].double(), rot[:, None, :, 1].double()
            a, b = y[..., :rot_dims // 2].clone(), y[..., rot_dims // 2:rot_dims].clone()
            y[..., :rot_dims // 2], y[..., rot_dims // 2:rot_dims] = a * c - b * s, b * c + a * s
        return y
    ones = torch.ones(dim, device=DEV)
    for blended in (False, True):
        k_cache = torch.zeros((12, kv_heads, page, dim), dtype=act, device=DEV)
        v_cache = torch.zeros((12, kv_heads, page, vdim), dtype=act, device=DEV)
        keep = torch.zeros((tokens, nv + 8), dtype=act, device=DEV)
        xd = x.to(DEV)
        ops.head_norm_rope_cache(xd, 0, nq, nq + nk, heads, kv_heads, dim, vdim, ones, ones, 1e-5, None if rot is None else rot.to(DEV),
                                 rot_dims, "half", slots.to(DEV), k_cache, v_cache, page, bias=bias.to(DEV), keep=keep[:, :nv],
                                 blend=(first.to(DEV), share) if blended else None)
        close(xd[:, :nq].view(tokens, heads, dim), turned(biased[:, :nq].view(tokens, heads, dim)), dtype, "q", bound=tight(dtype))
        values = biased[:, nq + nk:]
        close(keep[:, :nv], values, dtype, "kept values", bound=tight(dtype))
        assert not keep[:, nv:].any()
        if blended:
            values = (1 - share) * values + share * first.double()
        flat_k = k_cache.permute(0, 2, 1, 3).reshape(-1, kv_heads, dim).cpu()
        flat_v = v_cache.permute(0, 2, 1, 3).reshape(-1, kv_heads, vdim).cpu()
        written = [int(s) for s in slots if s >= 0]
        at = [i for i, s in enumerate(slots.tolist()) if s >= 0]
        close(flat_k[written], turned(biased[:, nq:nq + nk].view(tokens, kv_heads, dim))[at], dtype, "keys in the pages", bound=tight(dtype))
        close(flat_v[written], values.view(tokens, kv_heads, vdim)[at], dtype, "values in the pages", bound=tight(dtype))
        untouched = sorted(set(range(12 * page)) - set(written))
        assert not flat_k[untouched].any() and not flat_v[untouched].any()


@pytest.mark.parametrize("experts, identity, top, groups, keep", [(8, 4, 3, 4, 2), (6, 0, 2, 1, 1), (3, 5, 8, 1, 1), (60, 4, 7, 8, 3), (1, 1, 1, 2, 1),
                                                                  (5, 1, 2, 6, 2), (90, 6, 40, 2, 1)])
@pytest.mark.parametrize("score", ["softmax", "sigmoid"])
def test_router_with_a_correction_and_identity_experts(experts, identity, top, groups, keep, score):
    """Ranks below zero everywhere, groups ranked by their best, weights that are the scores themselves, the
    identity experts' sum, and their factor where rows still lack their norm."""
    from mrun_b200.kernels import ops
    gen = torch.Generator().manual_seed(experts * 7 + top)
    tokens, total = 150, experts + identity
    logits = torch.randn(tokens, total + 1, generator=gen) * 2
    logits[0, :total] -= 80.0
    logits[1, 0] += 60.0
    correction = torch.rand(total, generator=gen) * 2 - 3.5
    chosen = torch.empty((tokens, top), dtype=torch.int32, device=DEV)
    sums = torch.randint(1 << 28, 1 << 40, (tokens,), generator=gen)
    normed = ops.NormedRows(torch.empty((tokens, 96), dtype=torch.bfloat16, device=DEV), sums.to(DEV), 1e-5)
    weights, gate, unchanged = ops.route_grouped(logits.to(DEV), experts, top, groups, keep, 1, 1.0, chosen=chosen, score=score,
                                                 correction=correction.to(DEV), identity=identity, renormalize=False, handed_on=normed)
    assert torch.allclose(gate.cpu().double(), torch.sigmoid(logits[:, total].double()), atol=1e-6)
    scores = torch.softmax(logits[:, :total].double(), -1) if score == "softmax" else torch.sigmoid(logits[:, :total].double())
    router = {"top": top, "groups": {"count": groups, "keep": keep}}
    factor = torch.rsqrt(sums.double() * 2.0 ** -30 / 96 + 1e-5)
    assert (unchanged is None) == (identity == 0)
    for t in range(tokens):
        margin = []
        picks = plain.choose_experts(router, scores[t], correction.double(), margin)
        if min(margin, default=1.0) < 1e-6:
            continue
        assert sorted(chosen[t].tolist()) == sorted(e if e < experts else -1 for e, _ in picks), f"token {t}"
        dense, rest = torch.zeros(experts, dtype=F64), 0.0
        for e, w in picks:
            if e < experts:
                dense[e] = w
            else:
                rest += float(w) * float(factor[t])
        assert torch.allclose(weights[t].cpu().double(), dense, rtol=2e-5, atol=1e-9), f"token {t}"
        if identity:
            assert float(unchanged[t]) == pytest.approx(rest, rel=1e-4, abs=1e-12)


def test_router_survives_logits_that_are_no_numbers():
    """No rank is ever above the least one: nothing is chosen, nothing outside the arrays is touched."""
    from mrun_b200.kernels import ops
    logits = torch.full((5, 9), float("nan"), device=DEV)
    logits[2] = torch.arange(9.0)
    for score in ("softmax", "sigmoid"):
        chosen = torch.full((5, 2), 77, dtype=torch.int32, device=DEV)
        weights, _, _ = ops.route_grouped(logits, 6, 2, 4, 2, 1, 1.0, chosen=chosen, score=score, identity=2, renormalize=False,
                                          correction=torch.zeros(8, device=DEV))
        assert chosen[[0, 1, 3, 4]].tolist() == [[-1, -1]] * 4 and not weights[[0, 1, 3, 4]].any()
        assert chosen[2].tolist() == [-1, -1]                # the last two of eight: identity experts


# ------------------------------------------------------------------ mixers alone

def enlivened(w, seed):
    return {k: lively("m." + k, v, seed).to(torch.bfloat16).float() for k, v in w.items()}


def latent_spec(hidden, m):
    from mrun_b200.config.spec import LatentAttentionSpec
    return LatentAttentionSpec(hidden=hidden, heads=m["heads"], dim=m["dim"], rot_dim=0, vdim=m["vdim"], q_rank=0, kv_rank=m["kv_rank"],
                               softmax_scale=m["scale"], eps=1e-5, head_gate=True)


LATENT_SHAPES = [(latent(3, 11, 7, 13, 0.5), 16), (latent(4, 32, 48, 64, 0.2), 16), (latent(6, 24, 16, 72, 0.25), 4), (latent(2, 64, 128, 128, 0.1), 8),
                 (latent(17, 8, 8, 48, 0.4), 8), (latent(2, 16, 32, 272, 0.06), 16), (latent(2, 64, 64, 512, 0.02), 16)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("m, page", LATENT_SHAPES)
def test_latent_attention_alone(dtype, m, page):
    from mrun_b200.parts import MIXERS
    rt = runtime(dtype, page)
    spec = latent_spec(48, m)
    w = random_tensors(MIXERS.tensor_specs(spec, "m"), "m", torch.Generator().manual_seed(m["dim"]))
    part = MIXERS.build(spec, w, rt)
    W = named(w, "m.")
    check_rows(lambda rows, ctx, caches: part.forward(rows, ctx, caches[0]), 48, dtype, LENGTHS,
               lambda h, _: plain.latent_attention(m, W, "m.", h, 1e-5), [part.cache_need()], rt)


@pytest.mark.parametrize("expand", [4, 0])
@pytest.mark.parametrize("dim, vdim, kv_rank, heads, page", [(64, 64, 80, 3, 16), (128, 128, 256, 2, 8), (128, 64, 40, 2, 4), (64, 128, 300, 5, 16)])
def test_latent_attention_with_keys_and_values_made(dim, vdim, kv_rank, heads, page, expand, monkeypatch):
    """Prompt portions whose keys and values are made from the contexts' latents, next to portions and single
    tokens that stay with the latent: one request in one piece and cut, and several side by side."""
    from mrun_b200.parts import MIXERS, latent_attention
    monkeypatch.setattr(latent_attention, "EXPAND_ROWS", expand)
    rt = runtime("bfloat16", page)
    m = latent(heads, dim, vdim, kv_rank, 1.5 / dim)
    spec = latent_spec(48, m)
    w = random_tensors(MIXERS.tensor_specs(spec, "m"), "m", torch.Generator().manual_seed(dim + vdim), std=0.2)
    part = MIXERS.build(spec, w, rt)
    made = []
    monkeypatch.setattr(part, "_expanded", lambda *a, inner=part._expanded: made.append(a[-1]) or inner(*a))
    W = named(w, "m.")
    total = 700
    gen = torch.Generator().manual_seed(2)
    x = torch.randn(total, 48, generator=gen).to(torch.bfloat16).float()
    want = plain.latent_attention(m, W, "m.", x.double(), 1e-5)
    for portions in ([total], [300, 400], [500, 1, 3, 2, 194], [128, 128, 127, 129, 188], [20, 40, 600, 5] + [1] * 35):
        close(run_cut(part, rt, x, portions, pages=-(-total // page) + 2), want, "bfloat16", f"portions {portions[:6]}")
    assert sorted(set(made)) == ([128, 256, 512, 1024] if expand else [])
    made.clear()
    lengths = {"a": 70, "b": 129, "c": 33, "d": 300, "e": 2}
    rows = {r: torch.randn(n + 20, 48, generator=gen).to(torch.bfloat16).float() for r, n in lengths.items()}
    book = Steps([part.cache_need()], rt, pages=1024 // page + 8, slots=5)
    fed = {r: 0 for r in rows}
    for sizes in ({"a": 60, "b": 120}, {"a": 10, "b": 9, "d": 300}, {"a": 1, "b": 1, "d": 1, "c": 33}, {"c": 7, "e": 2, "a": 9, "d": 1}):
        def run(ctx, places):
            h = torch.cat([rows[r][fed[r]:fed[r] + n] for r, n in sizes.items()]).to(DEV, torch.bfloat16)
            return part.forward(h, ctx, book.caches[0]).float().cpu()
        got, at = book.run([(r, [0] * n) for r, n in sizes.items()], run), 0
        for r, n in sizes.items():
            expected = plain.latent_attention(m, W, "m.", rows[r].double(), 1e-5)
            fed[r] += n
            close(got[at:at + n], expected[fed[r] - n:fed[r]], "bfloat16", f"{r} beside others", bound=4e-2)
            at += n
    assert bool(made) == bool(expand)


def attention_spec(hidden, m, mix=None):
    from mrun_b200.config.sebevik import SebevikConfig
    from dataclasses import replace
    return replace(SebevikConfig._attention(m, "", hidden, 1e-5, None), value_mix=mix)


def attention_weights(spec, seed, std=0.3):
    from mrun_b200.parts import MIXERS
    w = random_tensors(MIXERS.tensor_specs(spec, "m"), "m", torch.Generator().manual_seed(seed), std=std)
    if "vmix" in w:
        w["vmix"] = torch.tensor(0.375)
    return enlivened(w, seed)


ATTENTION_SHAPES = [
    (attention(6, 3, 24, 40, 0.2, 30, 8, 500.0), 16), (attention(5, 5, 11, 7, 0.5, 7, 10, 30.0), 4),
    (attention(4, 2, 64, 64, 0.15, 33, 64, 1e6), 16),        # bfloat16: tcgen05 prompt tiles and TMA decode
    (attention(4, 2, 64, 64, 0.15, None, 32), 16), (attention(2, 1, 128, 64, 0.09, 50, 128), 8), (attention(4, 1, 64, 128, 0.2, 64), 16),
    (attention(4, 2, 80, 48, 0.1, 21, 80, 300.0), 8),        # the mma.sync kernels
    (attention(3, 3, 32, 16, 0.4, 1, 16), 4), (attention(34, 2, 16, 16, 0.5, 90, 4), 16)]


@pytest.mark.parametrize("dtype, tensor_cores", [("float32", False), ("bfloat16", False), ("bfloat16", True)])
@pytest.mark.parametrize("m, page", ATTENTION_SHAPES)
def test_two_attentions_that_share_values(dtype, tensor_cores, m, page, monkeypatch):
    """A layer, the same layer as the first of those that blend values, and one that blends: all on the same
    rows, each with pages of its own."""
    from mrun_b200.parts import MIXERS, gated_attention
    monkeypatch.setattr(gated_attention, "TENSOR_CORES", tensor_cores)
    rt = runtime(dtype, page)
    hidden = 64
    parts, weights = [], []
    for seed, mix in ((1, None), (1, "first"), (2, "blend")):
        spec = attention_spec(hidden, m, mix)
        w = attention_weights(spec, seed + m["dim"])
        if mix == "first":
            w.update({k: v for k, v in weights[0].items()})
        weights.append(w)
        parts.append(MIXERS.build(spec, w, rt))
    if tensor_cores and not parts[0].tensor_cores:
        pytest.skip("the tensor-core kernels do not take this shape")

    def want(h, _):
        a, values = plain.attention(m, named(weights[1], "m."), "m.", h, 1e-5)
        b, _ = plain.attention(m, named(weights[2], "m."), "m.", h, 1e-5, values)
        unmixed, _ = plain.attention(m, named(weights[2], "m."), "m.", h, 1e-5)
        assert float((b - unmixed).abs().max() / b.abs().max()) > 0.05
        return torch.cat([a, a, b], dim=1)
    check_rows(lambda rows, ctx, caches: torch.cat([p.forward(rows, ctx, c) for p, c in zip(parts, caches)], dim=1), hidden, dtype,
               LENGTHS, want, [p.cache_need() for p in parts], rt)


@pytest.mark.parametrize("tma, tc5, cluster", [(True, True, True), (True, True, False), (False, False, False)])
@pytest.mark.parametrize("m", [attention(4, 2, 128, 128, 0.1, 400, 64), attention(8, 1, 64, 128, 0.15, None, 64), attention(2, 2, 128, 64, 0.1, 129),
                               attention(3, 3, 80, 48, 0.1, 700, 80)])
def test_long_context_on_every_tensor_core_kernel(m, tma, tc5, cluster, monkeypatch):
    """Keys and values of one and of two sizes, a sink a head, in one piece and cut, on the tcgen05 / TMA / cluster
    kernels and on the older ones; a handful of rows (the product's own epilogue) and more."""
    from mrun_b200.kernels import attention as kernels
    from mrun_b200.parts import MIXERS
    for name, value in (("TMA_DECODE", tma), ("TC5_PREFILL", tc5), ("CLUSTER_DECODE", cluster)):
        monkeypatch.setattr(kernels, name, value)
    rt = runtime("bfloat16", 16)
    spec = attention_spec(64, m)
    w = attention_weights(spec, 3)
    part = MIXERS.build(spec, w, rt)
    assert part.tensor_cores and part.fusable
    total = 1100
    x = torch.randn(total, 64, generator=torch.Generator().manual_seed(9)).to(torch.bfloat16).float()
    want, _ = plain.attention(m, named(w, "m."), "m.", x.double(), 1e-5)
    for portions in ([total], [1060] + [1] * 40, [500, 1, 300, 2, 257] + [1] * 40):
        close(run_cut(part, rt, x, portions, pages=-(-total // 16) + 2), want, "bfloat16", f"portions {portions[:6]}")


@pytest.mark.parametrize("requests", [3, 16, 17, 40])
def test_many_single_tokens_with_blended_values(requests):
    """A decode step of many requests: up to sixteen rows the product adds biases and blends, above that the
    kernel behind it does."""
    from mrun_b200.parts import MIXERS
    rt = runtime("bfloat16", 16)
    m = attention(4, 2, 64, 64, 0.15, 20, 64)
    specs = [attention_spec(64, m, "first"), attention_spec(64, m, "blend")]
    weights = [attention_weights(s, i) for i, s in enumerate(specs)]
    parts = [MIXERS.build(s, w, rt) for s, w in zip(specs, weights)]
    lengths = [1 + (7 * i) % 45 for i in range(requests)]
    gen = torch.Generator().manual_seed(requests)
    x = [torch.randn(n + 4, 64, generator=gen).to(torch.bfloat16).float() for n in lengths]
    book = Steps([p.cache_need() for p in parts], rt, pages=6 * requests, slots=requests)

    def step(places_rows):
        rows = torch.cat(places_rows).to(DEV, torch.bfloat16)
        return lambda ctx, places: torch.cat([p.forward(rows, ctx, c) for p, c in zip(parts, book.caches)], dim=1).float().cpu()
    for i, n in enumerate(lengths):
        book.run([(i, [0] * n)], step([x[i][:n]]))
    want = []
    for v in x:
        a, values = plain.attention(m, named(weights[0], "m."), "m.", v.double(), 1e-5)
        want.append(torch.cat([a, plain.attention(m, named(weights[1], "m."), "m.", v.double(), 1e-5, values)[0]], dim=1))
    for k in range(4):
        got = book.run([(i, [0]) for i in range(requests)], step([v[n + k:n + k + 1] for v, n in zip(x, lengths)]))
        close(got, torch.cat([w[n + k:n + k + 1] for w, n in zip(want, lengths)]), "bfloat16", f"decoded token {k}")


@pytest.mark.parametrize("dtype, tensor_cores", [("float32", False), ("bfloat16", False), ("bfloat16", True)])
@pytest.mark.parametrize("dim, vdim, size, page", [(24, 12, 21, 8), (64, 64, 37, 16), (128, 64, 64, 16), (20, 33, 16, 4), (80, 48, 50, 16)])
def test_one_key_at_the_edge_of_the_window_and_the_sink(dtype, tensor_cores, dim, vdim, size, page, monkeypatch):
    """One key and the queries that look for it are made so that its score dominates a head: at the first token,
    on both sides of a page border and far into the request.  The query on the last position that still
    sees it takes its value, the one further on does not; asked from inside a prompt portion, by tokens
    decoded alone and from portions of two and three tokens.  Then queries that score far below zero: the
    head with the high sink gives next to nothing, the one with the low sink its usual output."""
    from mrun_b200.parts import MIXERS, gated_attention
    monkeypatch.setattr(gated_attention, "TENSOR_CORES", tensor_cores)
    rt = runtime(dtype, page)
    hidden, heads = 32, 2
    m = attention(heads, 1, dim, vdim, 18.0 / dim, size, 8, 100.0)
    spec = attention_spec(hidden, m)
    w = attention_weights(spec, 17 + dim, std=0.1)
    w = {k: (v * 0.2 if k.endswith(".b") else v) for k, v in w.items()}
    w["q"][:, :2] = 0; w["k"][:, :2] = 0; w["v"][:, 1] = 0
    for row in (dim - 1, 2 * dim - 1):                  # the last, unrotated feature of both heads' queries reads input column 1
        w["q"][row] = 0; w["q"][row, 1] = 1
    w["k"][dim - 1] = 0; w["k"][dim - 1, 0] = 1         # and the key's column 0
    w["sink"] = torch.tensor([4.0, -40.0])
    part = MIXERS.build(spec, w, rt)
    if tensor_cores and not part.tensor_cores:
        pytest.skip("the tensor-core kernels do not take this shape")
    W = named(w, "m.")
    total = 5 * size + 40
    gen = torch.Generator().manual_seed(3)
    reference = lambda x, W=W: plain.attention(m, W, "m.", x.to(rt.precision.act).double(), 1e-5)[0]
    for far in (0, page - 1, page, 3 * size + 3):
        last_seen = far + size - 1
        x = torch.randn(total, hidden, generator=gen) * 0.5
        x[:, :2] = 0
        x[far, 0] = 30.0
        inside, outside = sorted({min(far + 1, last_seen), last_seen}), [last_seen + 1, last_seen + 2]
        x[inside + outside, 1] = 30.0
        want = reference(x)
        lost = x.clone(); lost[far, 0] = 0
        change = (want - reference(lost)).abs().max(1).values / want.abs().max()
        assert float(change[inside].min()) > 0.2 and float(change[outside].max()) == 0.0
        for portions in edge_cuts(total, last_seen + 1):
            got = run_cut(part, rt, x, portions, pages=-(-total // page) + 2)
            what = f"key at {far}, last seen at {last_seen}, portions {portions[:8]}"
            close(got[inside + outside], want[inside + outside], dtype, what + ": the queries at the edge")
            close(got, want, dtype, what + ": all tokens")
    x = torch.randn(total, hidden, generator=gen) * 0.5
    x[:, 0] = 2.0; x[:, 1] = 0
    deniers = [0, 1, size, 2 * size + 5, total - 4, total - 1]
    x[deniers, 1] = -30.0
    want = reference(x)
    for shifted in (torch.tensor([-40.0, -40.0]), torch.tensor([4.0, 4.0]), torch.tensor([-40.0, 4.0])):
        change = (want - reference(x, dict(W, **{"m.sink": shifted.double()}))).abs().max(1).values / want.abs().max()
        assert float(change[deniers].min()) > 0.02
    for portions in ([total], [total - 6] + [1] * 6, edge_cuts(total, size)[2]):
        close(run_cut(part, rt, x, portions, pages=-(-total // page) + 2), want, dtype, f"the sinks, portions {portions[:8]}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim, kv_rank, page", [(16, 40, 8), (32, 64, 16), (24, 272, 4)])
def test_latent_attention_finds_one_far_key(dtype, dim, kv_rank, page):
    """One latent channel carries the key, the heads' key up-projections pass it to their last feature, and the
    queries that look for it, hundreds of tokens later, are large there."""
    from mrun_b200.parts import MIXERS
    rt = runtime(dtype, page)
    hidden, heads = 32, 2
    m = latent(heads, dim, 12, kv_rank, 0.5)
    spec = latent_spec(hidden, m)
    w = random_tensors(MIXERS.tensor_specs(spec, "m"), "m", torch.Generator().manual_seed(dim), std=0.1)
    w["q"][:, :2] = 0; w["dkv"][:, :2] = 0; w["g"][:, :2] = 0
    w["dkv"][kv_rank - 1] = 0; w["dkv"][kv_rank - 1, 0] = 1
    for row in (dim - 1, 2 * dim - 1):
        w["q"][row] = 0; w["q"][row, 1] = 1
        w["uk"][row] = 0; w["uk"][row, kv_rank - 1] = 1
    w["uv"][:, kv_rank - 1] = 1.0
    part = MIXERS.build(spec, w, rt)
    W = named(w, "m.")
    total = 360
    gen = torch.Generator().manual_seed(4)
    for far in (0, page - 1, page, 130):
        x = torch.randn(total, hidden, generator=gen) * 0.5
        x[:, :2] = 0
        x[far, 0] = 30.0
        asking = sorted({far + 1, far + 31, 200, 345, 359})
        x[asking, 1] = 20.0
        x = x.to(rt.precision.act).float()
        want = plain.latent_attention(m, W, "m.", x.double(), 1e-5)
        lost = x.clone(); lost[far, 0] = 0
        change = (want - plain.latent_attention(m, W, "m.", lost.double(), 1e-5)).abs().max(1).values / want.abs().max()
        assert float(change[asking].min()) > 0.1
        for portions in edge_cuts(total, 346):
            got = run_cut(part, rt, x, portions, pages=-(-total // page) + 2)
            close(got[asking], want[asking], dtype, f"key at {far}, portions {portions[:8]}: the queries that look for it")
            close(got, want, dtype, f"key at {far}, portions {portions[:8]}: all tokens")


def scan_spec(hidden, m):
    from mrun_b200.config.spec import SelectiveScanSpec
    return SelectiveScanSpec(hidden=hidden, inner=m["inner"], state=m["state"], dt_rank=m["dt_rank"], conv=m["conv"])


def scan_weights(spec, seed):
    from mrun_b200.parts import MIXERS
    w = random_tensors(MIXERS.tensor_specs(spec, "m"), "m", torch.Generator().manual_seed(seed))
    return enlivened(w, seed)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("m", [mamba1(48, 16, 8, 4), mamba1(37, 5, 3, 1), mamba1(128, 8, 32, 2), mamba1(60, 40, 12, 3), mamba1(100, 64, 33, 8),
                               mamba1(12, 130, 1, 4), mamba1(8, 256, 6, 2), mamba1(33, 1, 2, 5), mamba1(200, 32, 64, 4)])
def test_selective_scan_alone(dtype, m):
    from mrun_b200.parts import MIXERS
    rt = runtime(dtype)
    spec = scan_spec(48, m)
    w = scan_weights(spec, m["inner"] + m["state"])
    part = MIXERS.build(spec, w, rt)
    W = named(w, "m.")
    check_rows(lambda rows, ctx, caches: part.forward(rows, ctx, caches[0]), 48, dtype, LENGTHS,
               lambda h, _: plain.mamba1(m, W, "m.", h), [part.cache_need()], rt)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("inner, states", [(24, 16), (10, 3), (64, 100)])
def test_selective_scan_keeps_a_far_input_by_state(dtype, inner, states):
    """State 0 of channel 0 never decays, state 1 forgets at once: an input written into both is read from state
    0 hundreds of tokens later by the tokens whose C points at it, and is gone from state 1."""
    from mrun_b200.parts import MIXERS
    rt = runtime(dtype)
    hidden = 32
    m = mamba1(inner, states, 2, 2)
    spec = scan_spec(hidden, m)
    w = scan_weights(spec, 5)
    w = {k: (v * 0.1 if k in ("in", "x", "dt") else v) for k, v in w.items()}
    w["in"][:, :4] = 0
    for channel, column in ((0, 0), (1, 1), (2, 2)):        # channel 0: what is written; 1 and 2: what asks
        w["in"][channel] = 0; w["in"][channel, column] = 1
    w["conv"][:3, 0] = 0; w["conv"][:3, 1] = 1; w["conv.b"][:3] = 0
    w["in"][inner] = 0; w["in"][inner, 3] = 1               # channel 0's gate reads column 3, which is 4 everywhere
    R = 2
    w["x"][:, :3] = 0
    w["x"][R, 0] = w["x"][R + 1, 0] = 1                     # B_0 and B_1 read channel 0
    w["x"][R + states] = 0; w["x"][R + states, 1] = 1       # C_0 reads channel 1
    w["x"][R + states + 1] = 0; w["x"][R + states + 1, 2] = 1
    w["dt"][0] = 0; w["dt.b"][0] = 1.0
    w["A_log"][0, 0], w["A_log"][0, 1] = -60.0, 6.0
    w["o"] = w["o"] * 0.1
    w["o"][:, 0] = 1.0
    part = MIXERS.build(spec, w, rt)
    W = named(w, "m.")
    total = 420
    x = torch.randn(total, hidden, generator=torch.Generator().manual_seed(8)) * 0.3
    x[:, :3] = 0; x[:, 3] = 4.0
    x[5, 0] = 4.0
    keepers, forgetters = [6, 130, 300, 401, 419], [131, 402]
    x[keepers, 1] = 4.0
    x[forgetters, 2] = 4.0
    x = x.to(rt.precision.act).float()
    want = plain.mamba1(m, W, "m.", x.double())
    lost = x.clone(); lost[5, 0] = 0
    change = (want - plain.mamba1(m, W, "m.", lost.double())).abs().max(1).values / want.abs().max()
    assert float(change[keepers].min()) > 0.1 and float(change[forgetters].max()) < 1e-3
    for portions in ([total], [400] + [1] * 20, [3, 2, 2, 100, 193, 100] + [1] * 20, [31, 33, 32, 4, 5] + [2] * 150 + [15]):
        got = run_cut(part, rt, x, portions, pages=8)
        close(got[keepers], want[keepers], dtype, "the tokens that ask")
        close(got, want, dtype, "all tokens")


def test_selective_scan_over_a_long_request_of_slow_decays():
    """Thousands of tokens with decays next to one: the 32-bit path keeps their digits."""
    from mrun_b200.parts import MIXERS
    rt = runtime("float32")
    m = mamba1(16, 16, 4, 4)
    spec = scan_spec(24, m)
    w = scan_weights(spec, 2)
    w["A_log"] = w["A_log"] - 4.0
    w["dt.b"] = w["dt.b"] - 2.0
    part = MIXERS.build(spec, w, rt)
    x = torch.randn(4000, 24, generator=torch.Generator().manual_seed(1)) + 0.5
    want = plain.mamba1(m, named(w, "m."), "m.", x.double())
    close(run_cut(part, rt, x, [3990] + [1] * 10, pages=600), want, "float32", "slow decays", bound=1e-5)


# ------------------------------------------------------------------ the routed feed-forward alone

def routed_spec(hidden, mlp):
    from mrun_b200.config.sebevik import SebevikConfig
    return SebevikConfig._feed_forward({"mlp": mlp}, "", hidden)


@pytest.mark.parametrize("dtype, sort", [("float32", False), ("bfloat16", False), ("bfloat16", True)])
@pytest.mark.parametrize("hidden, mlp", [(64, moe(6, 2, 16, identity=2, groups=4, keep=2, shared=24)), (37, moe(3, 2, 7, identity=1)),
                                         (96, moe(4, 6, 32, identity=2, shared=32)), (64, moe(2, 1, 8, identity=6, groups=2, keep=1)),
                                         (40, moe(8, 3, 8, groups=2, keep=1, shared=8))])
@pytest.mark.parametrize("rows", [1, 16, 60])
def test_routed_feed_forward_alone(dtype, sort, hidden, mlp, rows, monkeypatch):
    """A token whose experts are all identity experts, one with none and everything between; on all experts
    with zero weights and on the chosen ones sorted; plain rows and rows that still lack their norm."""
    from mrun_b200.kernels import ops
    from mrun_b200.parts import FEED_FORWARDS, routed
    monkeypatch.setattr(routed, "SORT_MIN_SAVED_FLOPS", 0.0 if sort else 1e30)
    rt = runtime(dtype)
    spec = routed_spec(hidden, mlp)
    w = enlivened(random_tensors(FEED_FORWARDS.tensor_specs(spec, "m"), "m", torch.Generator().manual_seed(hidden)), 3)
    part = FEED_FORWARDS.build(spec, w, rt)
    W = named(w, "m.")
    x = torch.randn(rows, hidden, generator=torch.Generator().manual_seed(rows)).to(rt.precision.act)
    margins = []
    want = plain.routed_feed_forward(mlp, W, "m.", x.double(), margins)
    sure = margins[0] > (1e-4 if dtype == "float32" else 1e-2)
    assert int(sure.sum()) >= max(1, rows // 2)
    got = part.forward(x.to(DEV), None)
    close(got[sure], want[sure], dtype, "rows")
    pending = part.forward(x.to(DEV), None, defer_output=True)
    pending = pending.compute(torch.float32) if isinstance(pending, ops.PENDING) else pending
    close(pending[sure], want[sure], dtype, "rows left pending")
    if dtype == "bfloat16" and rows <= 16 and hidden % 32 == 0:
        scale = 2.5                                   # rows that are 1 / scale of what the product before made of them
        sums = torch.full((16,), round((1 / scale ** 2) * hidden * 2 ** 30), dtype=torch.int64, device=DEV)
        unfinished = ops.NormedRows((x.float() / scale).to(torch.bfloat16).to(DEV), sums, 0.0)
        close(part.forward(unfinished, None)[sure], want[sure], dtype, "rows that lack their norm")


# ------------------------------------------------------------------ whole models

@pytest.fixture(scope="module", params=sorted(STINY))
def stiny(request, tmp_path_factory):
    name = request.param
    return name, make_folder(name, str(tmp_path_factory.mktemp(f"sebevik_{name}"))), STINY[name]


def plain_logits(cfg, weights, tokens):
    margins = []
    logits = plain.forward(cfg, weights, tokens, margins=margins).to(torch.float32).numpy()
    return logits, close_calls(margins, len(tokens))


def test_layers_of_the_plain_run_and_the_engine_agree(stiny):
    """The engine's 32-bit residual stream after every layer is the plain run's."""
    from mrun_b200.engine import StepEntry
    from mrun_b200.engine.loading import executor_from_folder
    from mrun_b200.kernels import ops
    name, folder, settings = stiny
    cfg, weights = load_folder(folder)
    tokens = tokens_of(cfg["vocab"], 41, seed=4)
    logits, layers = plain.forward(cfg, weights, tokens, want_layers=True)
    ex = executor_from_folder(folder, dtype="float32", page_size=settings["page_size"], num_pages=48, max_requests=1)
    seen = []
    for block in ex.model.blocks:
        def forward(resid, delta, ctx, cache, inner=block.forward):
            out = inner(resid, delta, ctx, cache)
            seen.append((resid + (out.compute() if isinstance(out, ops.PENDING) else out)).cpu().double())
            return out
        block.forward = forward
    got = ex.step([StepEntry(ex.admit("r"), tokens, list(range(41)))]).cpu().double()
    assert len(seen) == len(layers) == len(cfg["layers"])
    for i, layer in enumerate(seen):
        error = float((layer - layers[i]).abs().max() / layers[i].abs().max())
        assert error < 2e-5, f"{name}: after layer {i} ({cfg['layers'][i]['type']}): {error:.3e}"
    assert float((got - logits).abs().max() / logits.abs().max()) < 2e-5


@pytest.mark.parametrize("dtype, sorted_experts, tensor_cores", [("float32", False, False), ("bfloat16", False, False),
                                                                ("bfloat16", True, True)])
def test_every_cutting_matches_plain(stiny, dtype, sorted_experts, tensor_cores, tmp_path, monkeypatch):
    """Whole prompts, a prefix and then token by token, portions of changing size down to one and two
    tokens, and up to four requests side by side in a pool so small that pages and state slots are used
    again.  A bfloat16 run is held to the bound where no router's choice up to the position was a close
    call, and at four in five of all positions."""
    name, folder, settings = stiny
    cfg, weights = load_folder(folder)
    vocab = cfg["vocab"]
    requests = {f"r{i}": tokens_of(vocab, n, seed=200 + i) for i, n in enumerate(TRACE_LENGTHS)}
    both = {rid: plain_logits(cfg, weights, tokens) for rid, tokens in requests.items()}
    want = {rid: logits for rid, (logits, _) in both.items()}
    unsure = {rid: flags for rid, (_, flags) in both.items()}
    if name == "sure":
        assert not any(bool(f.any()) for f in unsure.values())
    b = TraceBuilder()
    cuts = {}

    def section(label):
        cuts[label] = len(b.where)
    section("whole")
    for rid in ("r0", "r1", "r3", "r5"):
        cut_whole(b, rid, requests[rid])
    section("decode_tail")
    cut_decode_tail(b, "r0", requests["r0"])
    cut_decode_tail(b, "r7", requests["r7"], tail=2)
    cut_decode_tail(b, "r5", requests["r5"], tail=200 if name == "tensor" else 40)          # long decoding
    section("portions")
    for k, rid in enumerate(("r2", "r4", "r5", "r3")):
        cut_portions(b, rid, requests[rid], SIZES[k:] + SIZES[:k])
    section("mixed")
    cut_mixed(b, requests, SIZES, live=4, seed=6)
    rounded = sorted((-(-n // 64) * 64 for n in TRACE_LENGTHS), reverse=True)
    monkeypatch.setenv("MRUN_MOE_SORT_MIN_FLOPS", "0" if sorted_experts else "1e30")
    monkeypatch.setenv("MRUN_GATED_ATTENTION_TENSOR_CORES", "1" if tensor_cores else "0")
    runner = TraceRunner(folder, dtype, str(tmp_path / "out"), sum(rounded[:4]), settings["page_size"], max_requests=4)
    try:
        runner.run(b.steps)
    finally:
        assert runner.close() == 0
    scale = max(float(np.max(np.abs(w))) for w in want.values())
    bound = 2e-5 if dtype == "float32" else 4e-2
    files, first_seen, held, every = {}, {}, {}, {}
    for index, (step, row, rid, position) in enumerate(b.where):
        if step not in files:
            files[step] = runner.logits(step, vocab)
        got = files[step][row]
        if dtype == "float32":
            seen = first_seen.setdefault((rid, position), (got, step))
            assert np.array_equal(seen[0], got), (f"{name}: request {rid}, position {position}: steps {seen[1]} and "
                                                  f"{step} differ in bits")
        label = [l for l in cuts if cuts[l] <= index][-1]
        error = float(np.max(np.abs(got - want[rid][position]))) / scale
        every.setdefault(label, []).append(error)
        if dtype == "float32" or not unsure[rid][position]:
            held.setdefault(label, []).append((error, step, rid, position))
    for label, found in held.items():
        worst = max(found)
        print(name, dtype, label, f"{worst[0]:.2e}", len(found), len(every[label]))
        assert worst[0] <= bound, f"{name}/{dtype}/{label}: {worst}"
    for label, errors in every.items():
        within = sum(e <= bound for e in errors)
        assert within >= 0.8 * len(errors), f"{name}/{dtype}/{label}: only {within} of {len(errors)} positions within {bound}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_matches_plain(stiny, dtype):
    """Greedy generation through ``Engine.generate``: the scheduler cuts prompts into portions of seven tokens
    beside decoded tokens of other requests, with four state slots for five requests."""
    from mrun_b200 import Engine
    name, folder, settings = stiny
    cfg, weights = load_folder(folder)
    prompts = [tokens_of(cfg["vocab"], n, seed=300 + n) for n in (1, 9, 40, 71, 5)]
    engine = Engine.from_folder(folder, dtype=dtype, page_size=settings["page_size"], context=512, max_batch_tokens=7, max_requests=4)
    results = engine.generate(prompts, max_tokens=10, ignore_eos=True)
    assert bool(engine.executor._graphs) == engine.executor.model.graph_safe
    for prompt, result in zip(prompts, results):
        assert result.finish_reason == "length" and len(result.tokens) == 10
        tokens = list(prompt)
        for n, token in enumerate(result.tokens):
            margins = []
            logits = plain.forward(cfg, weights, tokens, margins=margins)[-1]
            best = int(torch.argmax(logits))
            margin = 1e-3 if dtype == "float32" else 2 * 4e-2 * float(logits.abs().max())
            unsure = dtype == "bfloat16" and bool(close_calls(margins, len(tokens))[-1])
            assert token == best or unsure or float(logits[best] - logits[token]) < margin, \
                f"{name}: output token {n}: engine {token}, plain {best}, behind by {float(logits[best] - logits[token]):.4f}"
            tokens.append(token)
    engine.executor.cache.check_invariants()
    assert not engine.executor.cache.live


def test_captured_decode_steps_are_used():
    """Every tiny model decodes captured, the one with more than sixteen heads over one latent too."""
    from mrun_b200.parts import MIXERS
    safe = {}
    for name in STINY:
        for i, layer in enumerate(sconfig(name).to_spec().layers):
            w = {t.name[2:]: torch.zeros(t.shape) for t in MIXERS.tensor_specs(layer.mixer, "m")}
            safe[name, i] = MIXERS.build(layer.mixer, w, runtime("bfloat16")).graph_safe
    assert all(safe.values())


def test_command_line_random_then_run(tmp_path):
    """``mrun random`` writes a Sebevik folder from its config.json, ``mrun run`` generates with it."""
    import json
    import os
    import subprocess
    import sys
    root = os.path.normpath(os.path.join(os.path.dirname(os.path.abspath(__file__)), os.pardir))
    mrun = os.path.join(root, "bin", "mrun")
    run = lambda *args: subprocess.run([sys.executable, mrun, *args], capture_output=True, text=True, timeout=600)
    (tmp_path / "cfg.json").write_text(json.dumps(STINY["wide"]["config"]))
    folder = str(tmp_path / "model")
    made = run("random", folder, "--config", str(tmp_path / "cfg.json"), "--seed", "21", "--std", "0.1")
    assert made.returncode == 0, made.stderr
    cfg, weights = load_folder(folder)
    prompt = tokens_of(cfg["vocab"], 19, seed=8)
    result = run("run", folder, "--prompt", ",".join(map(str, prompt)), "--max-tokens", "6", "--dtype", "float32",
                 "--ignore-eos", "--context", "1K")
    assert result.returncode == 0, result.stderr
    tokens = list(prompt)
    for token in (int(t) for t in result.stdout.strip().split(",")):
        logits = plain.forward(cfg, weights, tokens)[-1]
        best = int(torch.argmax(logits))
        assert token == best or float(logits[best] - logits[token]) < 1e-3
        tokens.append(token)
    assert len(tokens) == 19 + 6 and "Sebevik" in result.stderr


# ------------------------------------------------------------------ layer sizes of a real model

def real_sizes(top):
    routed = moe(6, top, 512, identity=2, groups=4, keep=2 if top == 2 else 4, shared=512)
    a = attention(8, 2, 128, 128, 128 ** -0.5, 160, 128, 500000.0, True)
    return {"architecture": "Sebevik", "vocab": 4096, "width": 1024, "norm": {"eps": 1e-6}, "layers": [
        {"type": "mamba1", "mixer": mamba1(2048, 16, 64, 4), "mlp": {"kind": "dense", "ff": 2816}},
        {"type": "attention", "mixer": a, "mlp": routed},
        {"type": "latent_attention", "mixer": latent(8, 128, 128, 256, 128 ** -0.5), "mlp": routed},
        {"type": "attention", "mixer": dict(a, mask={"size": 100}), "mlp": None}]}


@pytest.mark.parametrize("dtype, sorted_experts, top", [("float32", False, 2), ("bfloat16", False, 8), ("bfloat16", True, 2)])
def test_real_layer_sizes(dtype, sorted_experts, top, tmp_path, monkeypatch):
    """A width of 1,024, heads of 128 (in bfloat16 the tcgen05 and TMA attention kernels), a latent of 256, 2,048
    channels of 16 states, six experts of 512 with two identity experts: a prompt whole and in portions,
    then decoded token by token, against the plain model."""
    from mrun_b200.config.sebevik import SebevikConfig
    from mrun_b200.engine import StepEntry
    from mrun_b200.engine.loading import executor_from_folder
    from mrun_b200.parts import routed
    from mrun_b200.weights import write_random_model
    monkeypatch.setattr(routed, "SORT_MIN_SAVED_FLOPS", 0.0 if sorted_experts else 1e30)
    folder = write_random_model(SebevikConfig.from_dict(real_sizes(top)), str(tmp_path / "real"), seed=7, std=0.03, norm_noise=0.1)
    cfg, weights = load_folder(folder)
    tokens = tokens_of(cfg["vocab"], 330, seed=77)
    margins = []
    want = plain.forward(cfg, weights, tokens, margins=margins).to(torch.float32)
    sure = torch.from_numpy(~close_calls(margins, len(tokens))) if dtype == "bfloat16" else torch.ones(330, dtype=torch.bool)
    ex = executor_from_folder(folder, dtype=dtype, page_size=16, num_pages=96, max_requests=2)
    seen = {}
    for label, portions in (("whole", [330]), ("portions", [200, 3, 65, 30] + [1] * 32)):
        request, at, got = ex.admit(label), 0, []
        for n in portions:
            got.append(ex.step([StepEntry(request, tokens[at:at + n], list(range(n)))]).cpu())
            at += n
        ex.release(request)
        got = torch.cat(got)
        errors = (got - want).abs().max(1).values / want.abs().max()
        print(dtype, sorted_experts, label, f"{float(errors.max()):.2e}", int(sure.sum()))
        if dtype == "float32":
            assert float(errors.max()) <= 2e-5, f"{label}: {float(errors.max()):.3e}"
            assert torch.equal(seen.setdefault("logits", got), got), "the cuttings differ in bits"
        else:
            assert not bool(sure.any()) or float(errors[sure].max()) <= 4e-2, f"{label}: {float(errors[sure].max()):.3e}"
            assert top == 2 or int(sure.sum()) == 330
            assert int((errors <= 4e-2).sum()) >= 0.7 * len(tokens), f"{label}: {int((errors <= 4e-2).sum())} of {len(tokens)} within the bound"
    ex.check()
