"""Sebevik without a GPU: the registry, the configuration read back from its own dictionary, its refusals, the
tensor names and shapes of every part, which constants reach which spec, the cache needs, the order of
features of a rotated head, and hand-worked values of the plain implementation's functions."""
from __future__ import annotations

import copy
import json
import math

import pytest
import torch

import plain_sebevik as plain
from tiny_sebevik import STINY, load_folder, make_folder, sconfig

F = torch.float64


def test_registry_resolves_the_architecture():
    from mrun_b200 import registry
    from mrun_b200.config.sebevik import SebevikConfig
    assert registry.resolve({"architecture": "Sebevik"}) is SebevikConfig
    assert "sebevik" in registry.supported()


@pytest.mark.parametrize("name", sorted(STINY))
def test_read_back_and_tensors(name):
    from mrun_b200.config.sebevik import SebevikConfig
    from mrun_b200.weights.loader import expected_tensors
    config, raw = sconfig(name), STINY[name]["config"]
    assert config.to_dict() == raw
    assert SebevikConfig.from_dict(json.loads(json.dumps(config.to_dict()))) == config
    spec = config.to_spec()
    spec.validate()
    names = {t.name: t.shape for t in expected_tensors(spec)}
    width, want = raw["width"], {}
    want["embed"], want["final.norm"] = (raw["vocab"], width), (width,)
    for i, layer in enumerate(raw["layers"]):
        p, m, mlp = f"l{i}", layer["mixer"], layer["mlp"]
        want[f"{p}.norm1"] = (width,)
        q = f"{p}.mix"
        if layer["type"] == "latent_attention":
            H, D, V, R = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
            want.update({f"{q}.q": (H * D, width), f"{q}.dkv": (R, width), f"{q}.dkv.norm": (R,), f"{q}.uk": (H * D, R),
                         f"{q}.uv": (H * V, R), f"{q}.g": (H, width), f"{q}.o": (width, H * V)})
        elif layer["type"] == "attention":
            H, D, V = m["heads"], m["dim"], m["vdim"]
            G = m.get("kv_heads") or H
            for s, n in (("q", H * D), ("k", G * D), ("v", G * V)):
                want[f"{q}.{s}"], want[f"{q}.{s}.b"] = (n, width), (n,)
            want[f"{q}.sink"], want[f"{q}.o"] = (H,), (width, H * V)
            if m.get("v_mix"):
                want[f"{q}.vmix"] = ()
        else:
            I, N, R = m["inner"], m["state"], m["dt_rank"]
            want.update({f"{q}.in": (2 * I, width), f"{q}.conv": (I, m["conv"]), f"{q}.conv.b": (I,), f"{q}.x": (R + 2 * N, I),
                         f"{q}.dt": (I, R), f"{q}.dt.b": (I,), f"{q}.A_log": (I, N), f"{q}.D": (I,), f"{q}.o": (width, I)})
        if mlp is None:
            continue
        want[f"{p}.norm2"] = (width,)
        f = f"{p}.mlp"
        if mlp["kind"] == "dense":
            want[f"{f}.up"], want[f"{f}.down"] = (mlp["ff"], width), (width, mlp["ff"])
            continue
        ranked = mlp["router"]["experts"] + mlp["router"].get("identity", 0)
        want[f"{f}.router"], want[f"{f}.correction"] = (ranked, width), (ranked,)
        experts = [(f"e{e}", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
        if mlp.get("shared"):
            experts.append(("shared", mlp["shared"]["ff"]))
            want[f"{f}.shared.sg"] = (1, width)
        for e, ff in experts:
            want[f"{f}.{e}.gate"] = want[f"{f}.{e}.up"] = (ff, width)
            want[f"{f}.{e}.down"] = (width, ff)
    assert names == want
    assert config.num_parameters() == sum(math.prod(s) for s in want.values())


def test_constants_reach_the_parts():
    spec = sconfig("wide").to_spec()
    assert spec.tie_embeddings and all(l.arrangement == "pre_norm" for l in spec.layers)
    assert all(l.mixer_norm.offset == 1.0 and l.mixer_norm.eps == 1e-6 for l in spec.layers) and spec.final_norm.offset == 1.0
    plain_values, a, b = (spec.layers[i].mixer for i in (0, 2, 4))
    assert [s.value_mix for s in (plain_values, a, b)] == [None, "first", "blend"]       # the first layer that mixes, not the first
    assert (a.window, a.position.dims, a.position.base, a.position.pairing) == (20, 32, 10000.0, "interleaved")
    assert a.biases and a.sink and a.learned_sink and a.qk_norm == "unit" and not a.head_gate and a.softmax_scale == 0.2
    assert b.position is None and (b.heads, b.kv_heads, b.dim, b.vdim, b.window) == (6, 2, 16, 48, 64)
    latent = spec.layers[1].mixer
    assert latent.head_gate and (latent.rot_dim, latent.q_rank, latent.kv_rank, latent.window) == (0, 0, 72, None)
    scan = spec.layers[3].mixer
    assert (scan.inner, scan.state, scan.dt_rank, scan.conv) == (60, 40, 12, 2)
    routed = spec.layers[1].feed_forward
    assert (routed.experts, routed.identity, routed.top, routed.groups, routed.keep_groups, routed.group_top) == (7, 5, 2, 4, 1, 1)
    assert routed.score == "softmax" and routed.correction and not routed.renormalize and routed.route_scale == 1.0
    assert routed.shared_ff == 16 and routed.shared_gate
    plain_router = spec.layers[3].feed_forward
    assert (plain_router.groups, plain_router.identity, plain_router.shared_ff) == (1, 4, 0)
    assert sconfig("far").to_spec().layers[3].mixer.kv_heads == 3          # left out: one a query head
    assert sconfig("far").to_spec().layers[4].mixer.window is None


@pytest.mark.parametrize("name, path, value, message", [
    ("odd", ("width",), None, "width"), ("odd", ("norm", "eps"), 0, "norm.eps"), ("odd", ("layers",), [], "layers"),
    ("odd", ("layers", 1, "type"), "mamba2", "layers[1].type"), ("odd", ("layers", 0, "mixer", "kv_heads"), 2, "layers[0].mixer.heads"),
    ("odd", ("layers", 0, "mixer", "rot", "dims"), 12, "layers[0].mixer.rot.dims"),
    ("odd", ("layers", 0, "mixer", "rot", "dims"), 5, "layers[0].mixer.rot.dims"),
    ("odd", ("layers", 0, "mixer", "mask", "size"), 0, "layers[0].mixer.mask.size"),
    ("odd", ("layers", 0, "mixer", "v_mix"), 1, "layers[0].mixer.v_mix"),
    ("odd", ("layers", 3, "mixer", "vdim"), 2, "layers[3].mixer.v_mix"),
    ("odd", ("layers", 2, "mixer", "kv_rank"), None, "layers[2].mixer.kv_rank"),
    ("odd", ("layers", 1, "mixer", "dt_rank"), 0, "layers[1].mixer.dt_rank"),
    ("odd", ("layers", 2, "mlp", "router", "groups", "count"), 4, "layers[2].mlp.router.groups.count"),
    ("odd", ("layers", 2, "mlp", "router", "groups", "keep"), 4, "layers[2].mlp.router.groups.keep"),
    ("odd", ("layers", 2, "mlp", "router", "top"), 5, "layers[2].mlp.router.top"),
    ("odd", ("layers", 0, "mlp", "shared", "ff"), 0, "layers[0].mlp.shared.ff"),
    ("odd", ("layers", 1, "mlp", "kind"), "gated", "layers[1].mlp.kind")])
def test_refusals_name_the_key(name, path, value, message):
    from mrun_b200.config import ConfigError
    from mrun_b200.config.sebevik import SebevikConfig
    cfg = copy.deepcopy(STINY[name]["config"])
    at = cfg
    for key in path[:-1]:
        at = at[key]
    if value is None:
        at.pop(path[-1])
    else:
        at[path[-1]] = value
    with pytest.raises(ConfigError) as error:
        SebevikConfig.from_dict(cfg)
    assert message in str(error.value)


def test_checkpoint_without_a_tensor_is_refused(tmp_path):
    from mrun_b200.weights.loader import WeightsError, bind_tensors
    _, weights = load_folder(make_folder("sure", str(tmp_path / "m")))
    spec = sconfig("sure").to_spec()
    bind_tensors(spec, weights)
    weights.pop("l0.mix.sink")
    weights["l0.mix.extra"] = torch.zeros(3)
    with pytest.raises(WeightsError) as error:
        bind_tensors(spec, weights)
    assert error.value.missing == ["l0.mix.sink"] and error.value.unexpected == ["l0.mix.extra"]


def test_cache_needs():
    from mrun_b200.cache.needs import FixedState, PagedKV, PagedLatent
    from mrun_b200.parts import MIXERS, Precision, Runtime
    runtime = Runtime(torch.device("cpu"), Precision.of("bfloat16"), 16)
    needs = []
    for layer in sconfig("wide").to_spec().layers:
        tensors = {t.name[2:]: torch.zeros(t.shape) for t in MIXERS.tensor_specs(layer.mixer, "m")}
        needs.append(MIXERS.build(layer.mixer, tensors, runtime).cache_need())
    assert needs[0] == PagedKV(3, 24, 18, value_dim=40) and needs[1] == PagedLatent(80, None)
    assert needs[2] == PagedKV(2, 80, 20, value_dim=48) and needs[4] == PagedKV(2, 16, 64, value_dim=48)
    assert needs[3] == (FixedState((60, 40), "float32", name="state"), FixedState((1, 60), "bfloat16", name="conv"))


def test_half_split_order_keeps_pairs():
    from mrun_b200.parts.gated_attention import half_split_order
    assert half_split_order(8, 6) == [0, 2, 4, 1, 3, 5, 6, 7]
    q = torch.randn(5, 1, 8, dtype=F)
    at = torch.arange(5)
    rot = {"base": 30.0, "dims": 6}
    turned = plain.rotate(q, at, rot)[:, 0]
    moved = q[:, 0, half_split_order(8, 6)]
    f = 30.0 ** (-2.0 * torch.arange(3, dtype=F) / 6) * at[:, None]
    half = torch.cat([moved[:, :3] * torch.cos(f) - moved[:, 3:6] * torch.sin(f), moved[:, 3:6] * torch.cos(f) + moved[:, :3] * torch.sin(f),
                      moved[:, 6:]], dim=1)
    assert torch.allclose(turned[:, half_split_order(8, 6)], half)


def test_specs_that_no_part_takes():
    from dataclasses import replace
    from mrun_b200.parts import FEED_FORWARDS, MIXERS, Precision, Runtime
    runtime = Runtime(torch.device("cpu"), Precision.of("float32"), 8)
    a = sconfig("odd").to_spec().layers[0].mixer
    r = sconfig("odd").to_spec().layers[2].feed_forward

    def build(registry, spec):
        tensors = {t.name[2:]: torch.zeros(t.shape) for t in registry.tensor_specs(spec, "m")}
        return registry.build(spec, tensors, runtime)
    build(MIXERS, a); build(FEED_FORWARDS, r)
    for bad in (replace(a, value_mix="second"), replace(a, sink=False), replace(a, qk_norm="projection")):
        with pytest.raises(ValueError):
            build(MIXERS, bad)
    for bad in (replace(r, groups=4), replace(r, score="logit", groups=1, keep_groups=1), replace(r, top=7), replace(r, score="other")):
        with pytest.raises(ValueError):
            build(FEED_FORWARDS, bad)


# ------------------------------------------------------------------ hand-worked values of the plain functions

def test_plain_softmax_with_a_sink_and_a_window():
    s = torch.log(torch.tensor([[1.0, 2.0, 3.0]], dtype=F))
    mask = torch.tensor([[True, True, False]])
    got = plain.sink_softmax(s, mask, torch.tensor(math.log(5.0), dtype=F))
    assert torch.allclose(got, torch.tensor([[1 / 8, 2 / 8, 0.0]], dtype=F))
    high = plain.sink_softmax(s - 2000.0, mask, torch.tensor(900.0, dtype=F))
    assert torch.isfinite(high).all() and float(high.abs().max()) == 0.0
    assert plain.seen(4, 2).tolist() == [[True, False, False, False], [True, True, False, False],
                                         [False, True, True, False], [False, False, True, True]]


def test_plain_router():
    scores = torch.tensor([0.1, 0.3, 0.05, 0.35, 0.15, 0.05], dtype=F)
    correction = torch.tensor([-1.0, -3.0, -1.0, -1.2, -2.0, -2.0], dtype=F)
    router = {"experts": 4, "identity": 2, "top": 2, "groups": {"count": 3, "keep": 1}}
    # ranks: -0.9, -2.7 | -0.95, -0.85 | -1.85, -1.95: the second group's best is the largest
    picked = plain.choose_experts(router, scores, correction)
    assert [e for e, _ in picked] == [3, 2] and [float(w) for _, w in picked] == pytest.approx([0.35, 0.05])
    assert [e for e, _ in plain.choose_experts({"experts": 4, "identity": 2, "top": 3}, scores, correction)] == [3, 0, 2]


def test_plain_scan():
    x = torch.tensor([[1.0], [2.0]], dtype=F)
    dt = torch.tensor([[0.5], [1.0]], dtype=F)
    A = torch.tensor([[-math.log(2.0), -math.log(4.0)]], dtype=F)
    B = torch.tensor([[1.0, 2.0], [3.0, 1.0]], dtype=F)
    C = torch.tensor([[1.0, 1.0], [2.0, -1.0]], dtype=F)
    got = plain.selective_scan(x, dt, A, B, C, torch.tensor([10.0], dtype=F))
    # S_0 = (0.5, 1); S_1 = (0.25 + 6, 0.25 + 2)
    assert got.flatten().tolist() == pytest.approx([1.5 + 10.0, 2 * 6.25 - 2.25 + 20.0])
    conv = plain.causal_conv(torch.tensor([[1.0], [2.0], [3.0]], dtype=F), torch.tensor([[10.0, 1.0]], dtype=F), torch.tensor([0.5], dtype=F))
    assert conv.flatten().tolist() == [1.5, 12.5, 23.5]
