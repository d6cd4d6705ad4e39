"""The Sebevik decoder in plain torch on the CPU in 64-bit, one function per mechanism, written from
the design's equations and sharing nothing with the engine.  Slow on purpose: attention as a full
score matrix, the selective scan as a token-by-token loop, experts one token at a time.

Notation: h is what a sublayer reads (already normed), W the checkpoint's tensors by name (64-bit),
p a tensor-name prefix ending in a dot, m / mlp the layer's ``mixer`` / ``mlp`` entry of config.json.
"""
from __future__ import annotations

import torch

F = torch.float64


def as_double(weights):
    return {k: (v.to(F) if v.is_floating_point() else v) for k, v in weights.items()}


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def offset_norm(x, w, eps):
    """The layers' norm: the stored weight lies around zero and 1 is added to it."""
    return unit_rms(x, eps) * (1.0 + w)


def silu(z):
    return z * torch.sigmoid(z)


def seen(T, size=None):
    """[T, T]: which keys j a token i sees: all up to itself, or the last ``size`` of them."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    mask = j <= i
    return mask if size is None else mask & (i - j < size)


# ------------------------------------------------------------------ latent attention

def latent_attention(m, W, p, h, eps):
    """Keys and values of every head are up-projections of one normed latent a token; no positions;
    a head's output is multiplied by the sigmoid of its gate row."""
    H, D, V, T = m["heads"], m["dim"], m["vdim"], h.shape[0]
    q = (h @ W[p + "q"].T).view(T, H, D)
    c = unit_rms(h @ W[p + "dkv"].T, eps) * W[p + "dkv.norm"]
    k = (c @ W[p + "uk"].T).view(T, H, D)
    v = (c @ W[p + "uv"].T).view(T, H, V)
    gate = torch.sigmoid(h @ W[p + "g"].T)
    mask = seen(T)
    out = torch.zeros(T, H, V, dtype=F)
    for head in range(H):
        s = (q[:, head] @ k[:, head].T) * float(m["scale"])
        out[:, head] = torch.softmax(s.masked_fill(~mask, float("-inf")), -1) @ v[:, head] * gate[:, head:head + 1]
    return out.reshape(T, H * V) @ W[p + "o"].T


# ------------------------------------------------------------------ attention with a window, a sink and mixed values

def rotate(x, positions, rot):
    """x: [T, heads, dim].  Pair i = features (2i, 2i + 1) of the first rot['dims'] features turns by
    the angle position * base^(-2i/dims)."""
    if rot is None or not rot.get("dims"):
        return x
    dims = rot["dims"]
    f = float(rot["base"]) ** (-2.0 * torch.arange(dims // 2, dtype=F) / dims)
    a = positions.to(F)[:, None] * f[None, :]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def sink_softmax(s, mask, sink):
    """exp(s_j) / (exp(sink) + sum over the visible j of exp(s_j)) along the last axis."""
    s = s.masked_fill(~mask, float("-inf"))
    top = s.max(-1, keepdim=True).values.clamp_min(float(sink))
    e = torch.exp(s - top)
    return e / (torch.exp(sink - top) + e.sum(-1, keepdim=True))


def attention(m, W, p, h, eps, first=None):
    """(output, values as projected).  ``first``: the values [T, kv_heads, vdim] of the first layer that
    mixes values, None in that layer itself and where the layer does not mix."""
    H, D, V, T = m["heads"], m["dim"], m["vdim"], h.shape[0]
    G = m.get("kv_heads") or H
    positions = torch.arange(T)
    project = lambda name, n, d: (h @ W[p + name].T + W[p + name + ".b"]).view(T, n, d)
    q = unit_rms(rotate(project("q", H, D), positions, m.get("rot")), eps)
    k = unit_rms(rotate(project("k", G, D), positions, m.get("rot")), eps)
    values = v = project("v", G, V)
    if first is not None:
        lam = W[p + "vmix"]
        v = (1.0 - lam) * v + lam * first
    mask = seen(T, (m.get("mask") or {}).get("size"))
    out = torch.zeros(T, H, V, dtype=F)
    for head in range(H):
        g = head // (H // G)
        out[:, head] = sink_softmax((q[:, head] @ k[:, g].T) * float(m["scale"]), mask, W[p + "sink"][head]) @ v[:, g]
    return out.reshape(T, H * V) @ W[p + "o"].T, values


# ------------------------------------------------------------------ selective scan

def causal_conv(x, w, b):
    """Per channel; the last tap meets the token itself, zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=F), x])
    return sum(padded[i:i + T] * w[:, i] for i in range(taps)) + b


def selective_scan(x, dt, A, B, C, D):
    """S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n; y_c = sum_n S[c, n] C_n + D_c x_c."""
    S = torch.zeros_like(A)
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * x[t]
    return y


def mamba1(m, W, p, h):
    inner, N, R = m["inner"], m["state"], m["dt_rank"]
    xz = h @ W[p + "in"].T
    x, z = xz[:, :inner], xz[:, inner:]
    x = silu(causal_conv(x, W[p + "conv"], W[p + "conv.b"]))
    dbc = x @ W[p + "x"].T
    dt = torch.nn.functional.softplus(dbc[:, :R] @ W[p + "dt"].T + W[p + "dt.b"], threshold=1e9)
    y = selective_scan(x, dt, -torch.exp(W[p + "A_log"]), dbc[:, R:R + N], dbc[:, R + N:], W[p + "D"])
    return (y * silu(z)) @ W[p + "o"].T


# ------------------------------------------------------------------ feed-forwards

def dense(W, p, h):
    return torch.relu(h @ W[p + "up"].T) ** 2 @ W[p + "down"].T


def expert(W, p, h):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def choose_experts(router, scores, correction, margin=None):
    """scores: [experts + identity] of one token -> [(expert, weight)] in the order of choice.
    ``margin``, a list, receives how far the choice was from another one."""
    n, top = scores.numel(), router["top"]
    choice = scores + correction
    allowed = torch.ones(n, dtype=torch.bool)
    groups = router.get("groups")
    if groups is not None:
        best = choice.view(groups["count"], -1).max(1).values
        ranked = best.sort(descending=True)
        allowed = torch.zeros(groups["count"], n // groups["count"], dtype=torch.bool)
        allowed[ranked.indices[:groups["keep"]]] = True
        allowed = allowed.reshape(-1)
        if margin is not None and groups["keep"] < groups["count"]:
            margin.append(float(ranked.values[groups["keep"] - 1] - ranked.values[groups["keep"]]))
    ranked = choice.masked_fill(~allowed, float("-inf")).sort(descending=True)
    if margin is not None and top < int(allowed.sum()):
        margin.append(float(ranked.values[top - 1] - ranked.values[top]))
    return [(e, scores[e]) for e in ranked.indices[:top].tolist()]


def routed_feed_forward(mlp, W, p, h, margins=None):
    """``margins``, a list, receives one tensor [T]: each token's smallest gap of choice."""
    router = mlp["router"]
    scores = torch.softmax(h @ W[p + "router"].T, -1)
    y = torch.zeros_like(h)
    gaps = torch.full((h.shape[0],), float("inf"), dtype=F)
    for t in range(h.shape[0]):
        margin = []
        for e, w in choose_experts(router, scores[t], W[p + "correction"], margin):
            y[t] += w * (expert(W, f"{p}e{e}.", h[t:t + 1])[0] if e < router["experts"] else h[t])
        if margin:
            gaps[t] = min(margin)
    if margins is not None:
        margins.append(gaps)
    if mlp.get("shared") is not None:
        y = y + torch.sigmoid(h @ W[p + "shared.sg"].T) * expert(W, p + "shared.", h)
    return y


def feed_forward(mlp, W, p, h, margins=None):
    if mlp["kind"] == "dense":
        return dense(W, p, h)
    return routed_feed_forward(mlp, W, p, h, margins)


# ------------------------------------------------------------------ the model

def forward(cfg, weights, tokens, want_layers=False, margins=None):
    """float64 logits [T, vocab] of one sequence (and the residual stream after every layer).
    ``margins``, a list, receives one tensor [T] for every routed feed-forward."""
    W = as_double(weights)
    eps = float(cfg["norm"]["eps"])
    x = W["embed"][torch.tensor(tokens, dtype=torch.long)]
    first, after = None, []
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        h = offset_norm(x, W[f"l{i}.norm1"], eps)
        if layer["type"] == "latent_attention":
            y = latent_attention(m, W, p, h, eps)
        elif layer["type"] == "attention":
            mixes = bool(m.get("v_mix"))
            y, values = attention(m, W, p, h, eps, first if mixes else None)
            if mixes and first is None:
                first = values
        elif layer["type"] == "mamba1":
            y = mamba1(m, W, p, h)
        else:
            raise ValueError(layer["type"])
        x = x + y
        if layer.get("mlp") is not None:
            x = x + feed_forward(layer["mlp"], W, f"l{i}.mlp.", offset_norm(x, W[f"l{i}.norm2"], eps), margins)
        after.append(x)
    logits = offset_norm(x, W["final.norm"], eps) @ W["embed"].T
    return (logits, torch.stack(after)) if want_layers else logits
