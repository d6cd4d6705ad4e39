"""Small Katadra configurations for the tests, none like another: both mixers in several sizes (grouped
and ungrouped heads, keys and values of equal and of different sizes, head sizes that the tensor-core
kernels take and sizes that fit no vector width, bias tables from two rows to more than the longest
distance, caps that bend the scores and caps that hardly touch them, temperatures that change at every
position and never, time mixings with one head and many, state-space mixers with one to eight taps,
one group and many), feed-forwards behind either mixer and none, layers that run another one's
weights, directly and through a third."""
from __future__ import annotations

import json
import os

import numpy as np


def left(heads, kv_heads, dim, vdim, scale, cap, rows, reach, coef=0.4, every=20):
    out = {"heads": heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": cap, "bias_rows": rows, "bias_max": reach,
           "q_temp": {"coef": coef, "every": every}}
    if kv_heads is not None:
        out["kv_heads"] = kv_heads
    return out


def right(heads, dim, rank):
    return {"heads": heads, "dim": dim, "rank": rank}


def parallel(a, b, scales=(1.0, 1.0), ff=None):
    return {"type": "parallel", "mixer": {"left": a, "right": b, "left_scale": scales[0], "right_scale": scales[1]},
            "mlp": dense(ff)}


def mamba2(heads, vdim, state, groups, conv, parts, ff=None):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": parts}, "mlp": dense(ff)}


def dense(ff):
    return None if ff is None else {"kind": "dense", "ff": ff}


def again(layers, *owners):
    """The layers followed by entries that run the owners' weights."""
    return layers + [dict(layers[o], weights_of=o) for o in owners]


KTINY = {
    # every kernel's element-by-element form: sizes that fit no vector width, one tap, one-row parts
    "odd": {"page_size": 8, "seed": 37, "std": 0.15, "norm_noise": 0.2, "config": {
        "architecture": "Katadra", "vocab": 83, "width": 37, "norm": {"eps": 1e-5},
        "layers": again([mamba2(3, 7, 9, 1, 1, 3, 19), parallel(left(3, 1, 11, 5, 0.4, 3.0, 8, 30, 0.8, 3.5), right(3, 13, 3), (0.9, 0.4))],
                        1, 0, 0)}},
    # heads the mma.sync kernels take, keys wider than values and the other way round; a chain of owners
    "wide": {"page_size": 4, "seed": 32, "std": 0.12, "norm_noise": 0.15, "config": {
        "architecture": "Katadra", "vocab": 190, "width": 72, "norm": {"eps": 1e-6},
        "layers": again([parallel(left(6, 3, 48, 16, 0.3, 20.0, 16, 100, 0.3, 64), right(3, 24, 8), (0.9, 0.7), 88),
                         mamba2(6, 20, 16, 3, 4, 2),
                         parallel(left(4, 4, 32, 80, 0.25, 6.0, 6, 40, 0.5, 1), right(2, 40, 5), (-0.5, 1.0))], 2)
        + [dict(mamba2(6, 20, 16, 3, 4, 2), weights_of=1), dict(mamba2(6, 20, 16, 3, 4, 2), weights_of=4)]}},
    # heads of 64 (tcgen05 prompt tiles, TMA decode), long bias table, feed-forward behind the state space
    "tensor": {"page_size": 16, "seed": 33, "std": 0.1, "norm_noise": 0.1, "config": {
        "architecture": "Katadra", "vocab": 301, "width": 96, "norm": {"eps": 1e-5},
        "layers": [mamba2(4, 48, 64, 2, 3, 1, 64),
                   parallel(left(4, 2, 64, 64, 0.125, 50.0, 32, 600, 0.2, 100), right(2, 64, 16), (0.8, 1.1), 160),
                   mamba2(8, 16, 20, 4, 8, 8)]}},
    # keys of 128, values of 64, one kv head; a table of two rows; temperatures off
    "mixed": {"page_size": 16, "seed": 34, "std": 0.1, "norm_noise": 0.1, "config": {
        "architecture": "Katadra", "vocab": 150, "width": 64, "norm": {"eps": 1e-4},
        "layers": again([parallel(left(3, 1, 128, 64, 0.09, 15.0, 2, 50, 0.0, 7), right(4, 16, 4), (1.0, 0.25), 40),
                         mamba2(2, 96, 130, 1, 2, 6)], 0)}},
    # values of 128 with keys of 64; seventeen query heads a kv head in heads of 16
    "groups": {"page_size": 8, "seed": 35, "std": 0.12, "norm_noise": 0.1, "config": {
        "architecture": "Katadra", "vocab": 120, "width": 80, "norm": {"eps": 1e-5},
        "layers": [parallel(left(5, None, 64, 128, 0.15, 8.0, 12, 24, 0.6, 11), right(5, 8, 2), (0.7, 0.7)),
                   parallel(left(34, 2, 16, 16, 0.5, 30.0, 10, 200, 0.25, 40), right(1, 70, 12), (1.2, 0.4), 96),
                   mamba2(10, 8, 8, 5, 4, 5)]}},
}


def kconfig(name: str):
    from mrun_b200.config.katadra import KatadraConfig
    return KatadraConfig.from_dict(KTINY[name]["config"])


def make_folder(name: str, folder: str) -> str:
    from mrun_b200.weights import write_random_model
    t = KTINY[name]
    return write_random_model(kconfig(name), folder, seed=t["seed"], std=t["std"], norm_noise=t["norm_noise"])


def load_folder(folder: str):
    """config.json as a dict and every tensor as stored."""
    from safetensors.torch import load_file
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    return cfg, dict(load_file(os.path.join(folder, "model.safetensors")))


def tokens_of(vocab: int, length: int, seed: int) -> list:
    return np.random.default_rng(seed).integers(0, vocab, size=length).tolist()
