"""Small Sebevik configurations for the tests, none like another: the three mixers in several sizes (heads that the
tensor-core kernels take and sizes that fit no vector width, keys and values of equal and of different
sizes, latents up to rows of their own kernel's width, windows of one token and windows longer than every
request, rotations of all, of some and of no features, selective scans with one to eight taps and two to
more than a hundred states), values blended across layers whose query heads and keys differ, routers with and without
groups, identity experts and a shared expert, a dense feed-forward and none behind every mixer."""
from __future__ import annotations

import json
import os

import numpy as np


def latent(heads, dim, vdim, kv_rank, scale):
    return {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale}


def attention(heads, kv_heads, dim, vdim, scale, window=None, rot_dims=None, base=10000.0, v_mix=None):
    out = {"heads": heads, "dim": dim, "vdim": vdim, "scale": scale}
    if kv_heads is not None:
        out["kv_heads"] = kv_heads
    if window is not None:
        out["mask"] = {"size": window}
    if rot_dims is not None:
        out["rot"] = {"base": base, "dims": rot_dims}
    if v_mix is not None:
        out["v_mix"] = v_mix
    return out


def mamba1(inner, state, dt_rank, conv):
    return {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, identity=None, groups=None, keep=None, shared=None):
    router = {"experts": experts, "top": top}
    if identity is not None:
        router["identity"] = identity
    if groups is not None:
        router["groups"] = {"count": groups, "keep": keep}
    out = {"kind": "moe", "router": router, "expert": {"ff": ff}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def layer(kind, mix, mlp):
    return {"type": kind, "mixer": mix, "mlp": mlp}


STINY = {
    # every kernel's element-by-element form: sizes that fit no vector width, one tap, five states
    "odd": {"page_size": 8, "seed": 41, "std": 0.15, "norm_noise": 0.2, "config": {
        "architecture": "Sebevik", "vocab": 83, "width": 37, "norm": {"eps": 1e-5},
        "layers": [layer("attention", attention(3, 1, 10, 9, 0.4, 11, 6, 50.0, True), moe(3, 2, 7, shared=5)),
                   layer("mamba1", mamba1(23, 5, 3, 1), dense(19)),
                   layer("latent_attention", latent(3, 11, 7, 13, 0.3), moe(4, 3, 6, identity=2, groups=3, keep=2)),
                   layer("attention", attention(2, 1, 4, 9, 0.7, 5, 4, 10.0, True), None),
                   layer("mamba1", mamba1(11, 2, 1, 4), moe(2, 1, 9, identity=1))]}},
    # heads of 64 (tcgen05 prompt tiles, TMA decode) and a latent of 64; all features rotated
    "tensor": {"page_size": 16, "seed": 43, "std": 0.1, "norm_noise": 0.2, "config": {
        "architecture": "Sebevik", "vocab": 257, "width": 96, "norm": {"eps": 1e-5},
        "layers": [layer("mamba1", mamba1(128, 16, 8, 4), moe(6, 3, 16, identity=2, groups=4, keep=2, shared=24)),
                   layer("attention", attention(4, 2, 64, 64, 0.15, 33, 64, 1000000.0, True), dense(96)),
                   layer("latent_attention", latent(4, 32, 48, 64, 0.2), None),
                   layer("attention", attention(4, 2, 64, 64, 0.12, 40, 32, 500.0, True), moe(5, 2, 24, identity=1, shared=8))]}},
    # keys wider than values on the mma.sync kernels; the first attention mixes nothing; another number of
    # query heads and another key size where values are blended; latent rows padded to their kernel's width; states on 16 lanes
    "wide": {"page_size": 4, "seed": 47, "std": 0.12, "norm_noise": 0.15, "config": {
        "architecture": "Sebevik", "vocab": 190, "width": 72, "norm": {"eps": 1e-6},
        "layers": [layer("attention", attention(6, 3, 24, 40, 0.3, 18, 8, 300.0, False), dense(88)),
                   layer("latent_attention", latent(6, 24, 16, 72, 0.25), moe(7, 2, 16, identity=5, groups=4, keep=1, shared=16)),
                   layer("attention", attention(4, 2, 80, 48, 0.2, 20, 32, 10000.0, True), None),
                   layer("mamba1", mamba1(60, 40, 12, 2), moe(4, 2, 12, identity=4)),
                   layer("attention", attention(6, 2, 16, 48, 0.25, 64, None, v_mix=True), moe(8, 2, 8, groups=2, keep=1))]}},
    # every expert of every routed layer is chosen, so that no choice is a close call and a bfloat16 run is
    # compared at every position; keys of 128 with values of 64; a window of one token
    "sure": {"page_size": 16, "seed": 53, "std": 0.1, "norm_noise": 0.2, "config": {
        "architecture": "Sebevik", "vocab": 128, "width": 64, "norm": {"eps": 1e-4},
        "layers": [layer("attention", attention(2, 1, 128, 64, 0.09, 24, 128, 20000.0, True), moe(3, 4, 16, identity=1, shared=16)),
                   layer("latent_attention", latent(2, 16, 32, 128, 0.3), moe(2, 4, 8, identity=2, groups=2, keep=2)),
                   layer("mamba1", mamba1(64, 128, 4, 3), dense(64)),
                   layer("attention", attention(4, 1, 16, 64, 0.4, 1, 16, 100.0, True), moe(2, 2, 16))]}},
    # a window longer than every request and none at all; seventeen heads over one latent; a latent wider than
    # the per-head-size kernels; 130 states, a step rank of 33, eight taps; kv_heads left out
    "far": {"page_size": 8, "seed": 59, "std": 0.12, "norm_noise": 0.1, "config": {
        "architecture": "Sebevik", "vocab": 70, "width": 48, "norm": {"eps": 1e-5},
        "layers": [layer("latent_attention", latent(17, 8, 8, 48, 0.4), dense(40)),
                   layer("mamba1", mamba1(40, 130, 33, 8), None),
                   layer("latent_attention", latent(3, 20, 12, 272, 0.3), moe(5, 2, 8, identity=1, groups=6, keep=4, shared=8)),
                   layer("attention", attention(3, None, 32, 32, 0.3, 1000, 24, 10000.0), moe(2, 2, 8, identity=2, shared=4)),
                   layer("attention", attention(4, 4, 16, 16, 0.5), None)]}},
}


def sconfig(name: str):
    from mrun_b200.config.sebevik import SebevikConfig
    return SebevikConfig.from_dict(STINY[name]["config"])


def lively(name: str, tensor, seed: int):
    """What the random-weights mode leaves small where a fault would hide: sinks and biases of some size,
    corrections that make every rank negative, steps and rates from slow to fast."""
    import torch
    gen = torch.Generator().manual_seed(seed + len(name))
    rand = lambda: torch.rand(tensor.shape, generator=gen)
    last = name.rsplit(".", 1)[-1]
    if last == "sink":
        out = rand() * 4 - 1
    elif last == "correction":
        out = rand() * 0.6 - 1.5
    elif name.endswith((".q.b", ".k.b", ".v.b")):
        out = torch.randn(tensor.shape, generator=gen) * 0.5
    elif name.endswith(".dt.b"):
        out = rand() * 4 - 4
    elif last == "A_log":
        out = rand() * 5 - 3.5
    else:
        return tensor
    return out.to(tensor.dtype)


def make_folder(name: str, folder: str) -> str:
    from mrun_b200.weights import write_random_model
    from safetensors.torch import load_file, save_file
    t = STINY[name]
    write_random_model(sconfig(name), folder, seed=t["seed"], std=t["std"], norm_noise=t["norm_noise"])
    path = os.path.join(folder, "model.safetensors")
    save_file({n: lively(n, w, t["seed"]) for n, w in load_file(path).items()}, path)
    return folder


def load_folder(folder: str):
    """config.json as a dict and every tensor as stored."""
    from safetensors.torch import load_file
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    return cfg, dict(load_file(os.path.join(folder, "model.safetensors")))


def tokens_of(vocab: int, length: int, seed: int) -> list:
    return np.random.default_rng(seed).integers(0, vocab, size=length).tolist()
