"""The Katadra decoder in plain torch on the CPU in 64-bit, one function per mechanism, written from
the design's equations and sharing nothing with the engine.  Slow on purpose: attention as a full
score matrix, both recurrences as token-by-token loops.

Notation: h is what a sublayer reads, W the checkpoint's tensors by name (64-bit), p a tensor-name
prefix ending in a dot, m the layer's ``mixer`` entry of config.json.
"""
from __future__ import annotations

import math

import torch

F = torch.float64


def as_double(weights):
    return {k: (v.to(F) if v.is_floating_point() else v) for k, v in weights.items()}


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def silu(x):
    return x * torch.sigmoid(x)


# ------------------------------------------------------------------ attention

def bucket(n, rows, reach):
    """The row of the bias table for a key n positions back: one row a distance in the first half
    of the table, logarithmic steps up to ``reach`` in the second half, the last row beyond."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(reach / half) * (rows - half)))


def distance_bias(table, T, reach):
    """[H, T, T]: the bias of query i and key j <= i (zero elsewhere)."""
    rows, H = table.shape
    out = torch.zeros(H, T, T, dtype=F)
    at = torch.tensor([bucket(n, rows, reach) for n in range(T)])
    for i in range(T):
        out[:, i, :i + 1] = table[at[i - torch.arange(i + 1)]].T
    return out


def temperature(positions, coef, every):
    return 1.0 + coef * torch.log(torch.floor((positions.to(F) + 1.0) / every) + 1.0)


def soft_cap(s, cap):
    return cap * torch.tanh(s / cap)


def causal_softmax(s):
    T = s.shape[-1]
    seen = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    s = torch.where(seen, s, torch.full_like(s, float("-inf")))
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def biased_scores(m, table, q, k, eps):
    """q [T, H, D], k [T, G, D] as projected -> scores [H, T, T] before the mask."""
    T, H, _ = q.shape
    G = k.shape[1]
    q = unit_rms(q, eps) * temperature(torch.arange(T), m["q_temp"]["coef"], m["q_temp"]["every"])[:, None, None]
    k = unit_rms(k, eps)
    s = torch.stack([q[:, h] @ k[:, h // (H // G)].T for h in range(H)]) * m["scale"]
    return soft_cap(s, m["softcap"]) + distance_bias(table, T, m["bias_max"])


def attention_heads(m, W, p, h, eps):
    """The gated heads, before the output projection: [T, H * V]."""
    H, D, V, T = m["heads"], m["dim"], m["vdim"], h.shape[0]
    G = m.get("kv_heads") or H
    q = (h @ W[p + "q"].T).view(T, H, D)
    k = (h @ W[p + "k"].T).view(T, G, D)
    v = (h @ W[p + "v"].T).view(T, G, V)
    weights = causal_softmax(biased_scores(m, W[p + "rel"], q, k, eps))
    out = torch.stack([weights[i] @ v[:, i // (H // G)] for i in range(H)], dim=1)
    return out.reshape(T, H * V) * torch.sigmoid(h @ W[p + "g"].T)


def biased_attention(m, W, p, h, eps):
    return attention_heads(m, W, p, h, eps) @ W[p + "o"].T


# ------------------------------------------------------------------ time mixing

def token_shift(h, mu):
    """h + (previous token's h - h) * mu, zeros before the first token."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]], dim=0)
    return h + (before - h) * mu


def bonus_recurrence(r, k, v, w, u):
    """r, k, w [T, H, D], v [T, H, V], u [H, D]: reads the state before the token's own write, the
    token's own write weighed by u; then the state decays and takes the write."""
    T, H, D = r.shape
    S = torch.zeros(H, D, v.shape[2], dtype=F)
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for t in range(T):
        write = k[t][:, :, None] * v[t][:, None, :]
        out[t] = ((S + u[:, :, None] * write) * r[t][:, :, None]).sum(1)
        S = w[t][:, :, None] * S + write
    return out


def time_mixing(m, W, p, h, eps):
    H, D, T = m["heads"], m["dim"], h.shape[0]
    mix = {s: token_shift(h, W[p + "mu." + s]) for s in "rkvgw"}
    r, k, v = ((mix[s] @ W[p + s].T).view(T, H, D) for s in "rkv")
    gate = silu(mix["g"] @ W[p + "g"].T)
    w = torch.exp(-torch.exp(torch.tanh(mix["w"] @ W[p + "w1"].T) @ W[p + "w2"].T + W[p + "w0"])).view(T, H, D)
    o = unit_rms(bonus_recurrence(r, k, v, w, W[p + "u"]), eps).reshape(T, H * D)
    return (o * W[p + "norm"] * gate) @ W[p + "o"].T


def parallel_mixer(m, W, p, h, eps):
    return (m["left_scale"] * biased_attention(m["left"], W, p + "left.", h, eps)
            + m["right_scale"] * time_mixing(m["right"], W, p + "right.", h, eps))


# ------------------------------------------------------------------ state-space mixer

def short_conv(x, w, b):
    """Causal convolution over time per channel: x [T, C], w [C, taps], the last column weighs the
    current token, zeros before the start; a bias; SiLU."""
    T, taps = x.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=F), x], dim=0)
    return silu(sum(padded[j:j + T] * w[:, j] for j in range(taps)) + b)


def state_space(x, B, C, dt, a_log):
    """x [T, H, V], B, C [T, G, N], dt [T, H] (positive): S <- exp(-e^a_log dt) S + dt B x^T,
    y = S^T C."""
    T, H, V = x.shape
    G, N = B.shape[1], B.shape[2]
    S = torch.zeros(H, N, V, dtype=F)
    y = torch.zeros(T, H, V, dtype=F)
    group = torch.arange(H) // (H // G)
    for t in range(T):
        decay = torch.exp(-torch.exp(a_log) * dt[t])
        S = decay[:, None, None] * S + dt[t][:, None, None] * B[t, group][:, :, None] * x[t][:, None, :]
        y[t] = (S * C[t, group][:, :, None]).sum(1)
    return y


def mamba2(m, W, p, h, eps):
    H, V, N, G, T = m["heads"], m["vdim"], m["state"], m["groups"], h.shape[0]
    inner = H * V
    z, xbc, dt = torch.split(h @ W[p + "in"].T, [inner, inner + 2 * G * N, H], dim=1)
    x, B, C = torch.split(short_conv(xbc, W[p + "conv"], W[p + "conv.b"]), [inner, G * N, G * N], dim=1)
    dt = torch.nn.functional.softplus(dt + W[p + "dt_bias"], threshold=1e9)
    x = x.reshape(T, H, V)
    y = state_space(x, B.reshape(T, G, N), C.reshape(T, G, N), dt, W[p + "A_log"])
    y = (y + W[p + "D"][None, :, None] * x).reshape(T, inner) * silu(z)
    y = unit_rms(y.view(T, m["norm_groups"], inner // m["norm_groups"]), eps).reshape(T, inner)
    return (y * W[p + "norm"]) @ W[p + "o"].T


# ------------------------------------------------------------------ layers and model

def dense_feed_forward(W, p, h):
    u = torch.relu(h @ W[p + "up"].T)
    return (u * u) @ W[p + "down"].T


def mixer(layer, W, p, h, eps):
    return {"parallel": parallel_mixer, "mamba2": mamba2}[layer["type"]](layer["mixer"], W, p, h, eps)


def forward(cfg, weights, tokens, want_layers=False):
    """float64 logits [T, vocab] of one sequence (and the residual stream after every layer run)."""
    W = as_double(weights)
    eps = float(cfg["norm"]["eps"])
    x = W["embed"][torch.tensor(tokens, dtype=torch.long)]
    after = []
    for i, layer in enumerate(cfg["layers"]):
        while layer.get("weights_of") is not None:      # another layer's weights, this layer's place in the order
            i = layer["weights_of"]
            layer = cfg["layers"][i]
        p = f"l{i}."
        x = x + layer_norm(mixer(layer, W, p + "mix.", x, eps), W[p + "norm1"], W[p + "norm1.b"], eps)
        if layer.get("mlp") is not None:
            x = x + layer_norm(dense_feed_forward(W, p + "mlp.", x), W[p + "norm2"], W[p + "norm2.b"], eps)
        after.append(x)
    logits = layer_norm(x, W["final.norm"], W["final.norm.b"], eps) @ W["head"].T
    return (logits, torch.stack(after)) if want_layers else logits
