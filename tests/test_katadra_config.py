"""Katadra without a GPU: the registry, the configuration read back from its own dictionary, its refusals,
the tensor names and shapes of every part, layers that share weights, the table over distances, the
random-weights folder, and hand-worked values of the plain implementation's functions."""
from __future__ import annotations

import copy
import json
import math
import os

import pytest
import torch

import plain_katadra as plain
from tiny_katadra import KTINY, kconfig, load_folder, make_folder

F = torch.float64


def test_registry_resolves_the_architecture():
    from mrun_b200 import registry
    from mrun_b200.config.katadra import KatadraConfig
    assert registry.resolve({"architecture": "Katadra"}) is KatadraConfig
    assert "katadra" in registry.supported()


@pytest.mark.parametrize("name", sorted(KTINY))
def test_read_back_and_spec(name):
    from mrun_b200.config.katadra import KatadraConfig
    from mrun_b200.weights.loader import expected_tensors
    config, raw = kconfig(name), KTINY[name]["config"]
    assert config.to_dict() == raw
    assert KatadraConfig.from_dict(json.loads(json.dumps(config.to_dict()))) == config
    spec = config.to_spec()
    names = {t.name: t.shape for t in expected_tensors(spec)}
    width = raw["width"]
    assert names["embed"] == names["head"] == (raw["vocab"], width)
    assert names["final.norm"] == names["final.norm.b"] == (width,)
    order = spec.run_order()
    assert len(order) == len(raw["layers"])
    for i, layer in enumerate(raw["layers"]):
        p, m = f"l{i}", layer["mixer"]
        owner = i
        while raw["layers"][owner].get("weights_of") is not None:
            owner = raw["layers"][owner]["weights_of"]
        assert spec.layers[order[i].layer].prefix == f"l{owner}" and order[i].cache_of is None
        if owner != i:
            assert not any(n.startswith(p + ".") for n in names)
            continue
        assert spec.layers[order[i].layer].arrangement == "post_norm"
        assert names[f"{p}.norm1"] == names[f"{p}.norm1.b"] == (width,)
        assert (f"{p}.norm2" in names) == (f"{p}.norm2.b" in names) == (layer["mlp"] is not None)
        if layer["mlp"]:
            assert names[f"{p}.mlp.up"] == (layer["mlp"]["ff"], width) and names[f"{p}.mlp.down"] == (width, layer["mlp"]["ff"])
        if layer["type"] == "parallel":
            a, r, q = m["left"], m["right"], f"{p}.mix.left"
            groups = a.get("kv_heads") or a["heads"]
            assert names[f"{q}.q"] == (a["heads"] * a["dim"], width) and names[f"{q}.k"] == (groups * a["dim"], width)
            assert names[f"{q}.v"] == (groups * a["vdim"], width) and names[f"{q}.g"] == (a["heads"] * a["vdim"], width)
            assert names[f"{q}.o"] == (width, a["heads"] * a["vdim"]) and names[f"{q}.rel"] == (a["bias_rows"], a["heads"])
            assert f"{q}.q.norm" not in names and f"{q}.out" not in names
            inner, q = r["heads"] * r["dim"], f"{p}.mix.right"
            for s in "rkvg":
                assert names[f"{q}.{s}"] == (inner, width) and names[f"{q}.mu.{s}"] == (width,)
            assert names[f"{q}.mu.w"] == (width,) and names[f"{q}.w1"] == (r["rank"], width)
            assert names[f"{q}.w2"] == (inner, r["rank"]) and names[f"{q}.w0"] == names[f"{q}.norm"] == (inner,)
            assert names[f"{q}.u"] == (r["heads"], r["dim"]) and names[f"{q}.o"] == (width, inner)
        else:
            inner, q = m["heads"] * m["vdim"], f"{p}.mix"
            channels = inner + 2 * m["groups"] * m["state"]
            assert names[f"{q}.in"] == (inner + channels + m["heads"], width)
            assert names[f"{q}.conv"] == (channels, m["conv"]) and names[f"{q}.conv.b"] == (channels,)
            assert names[f"{q}.dt_bias"] == names[f"{q}.A_log"] == names[f"{q}.D"] == (m["heads"],)
            assert names[f"{q}.norm"] == (inner,) and names[f"{q}.o"] == (width, inner)


def test_constants_reach_the_parts():
    spec = kconfig("odd").to_spec()
    mix = spec.layers[1].mixer
    a, r = mix.left, mix.right
    assert mix.combine == "sum" and mix.scales == (0.9, 0.4)
    assert a.temperature == (0.8, 3.5) and a.soft_cap == 3.0 and a.distance_bias == (8, 30.0) and a.softmax_scale == 0.4
    assert a.qk_norm == "unit" and a.element_gate and not a.sink and not a.head_gate and a.position is None and a.window is None
    assert (a.heads, a.kv_heads, a.dim, a.vdim) == (3, 1, 11, 5) and (r.heads, r.dim, r.rank) == (3, 13, 3)
    s = spec.layers[0].mixer
    assert (s.heads, s.vdim, s.state, s.groups, s.conv, s.norm_groups) == (3, 7, 9, 1, 1, 3)
    assert kconfig("groups").to_spec().layers[0].mixer.left.kv_heads == 5      # left out: one a query head
    assert all(part.eps == 1e-5 for part in (a, r, s, spec.final_norm, spec.layers[1].mixer_norm))


def test_sizes_that_only_the_checkpoint_gives(tmp_path):
    """The bias table's rows and the low-rank size are read from the tensors' shapes."""
    from mrun_b200 import registry
    folder = make_folder("wide", str(tmp_path / "m"))
    cfg, weights = load_folder(folder)
    for entry in cfg["layers"]:
        if entry["type"] == "parallel":
            entry["mixer"]["left"].pop("bias_rows"); entry["mixer"]["right"].pop("rank")
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    config = registry.load_config(folder)
    assert config.to_spec().layers == kconfig("wide").to_spec().layers
    assert config.num_parameters() == sum(t.numel() for t in weights.values())


@pytest.mark.parametrize("path, value, message", [
    (("width",), None, "width"), (("norm", "eps"), 0, "norm.eps"), (("layers",), [], "layers"),
    (("layers", 0, "type"), "mamba3", "layers[0].type"), (("layers", 0, "mixer", "groups"), 2, "layers[0].mixer.heads"),
    (("layers", 0, "mixer", "norm_groups"), 4, "layers[0].mixer.norm_groups"),
    (("layers", 0, "mlp", "kind"), "moe", "layers[0].mlp.kind"), (("layers", 1, "mixer", "left", "kv_heads"), 2, "layers[1].mixer.left.heads"),
    (("layers", 1, "mixer", "left", "softcap"), -1, "layers[1].mixer.left.softcap"),
    (("layers", 1, "mixer", "left", "q_temp", "every"), 0, "layers[1].mixer.left.q_temp.every"),
    (("layers", 1, "mixer", "left", "bias_rows"), None, "layers[1].mixer.left.bias_rows"),
    (("layers", 1, "mixer", "right", "rank"), None, "layers[1].mixer.right.rank"),
    (("layers", 1, "mixer", "left_scale"), "x", "layers[1].mixer.left_scale"),
    (("layers", 2, "weights_of"), 9, "layers[2].weights_of"), (("layers", 1, "weights_of"), 2, "weights_of")])
def test_refusals_name_the_key(path, value, message):
    from mrun_b200.config import ConfigError
    from mrun_b200.config.katadra import KatadraConfig
    cfg = copy.deepcopy(KTINY["odd"]["config"])
    if path == ("layers", 1, "weights_of"):
        cfg["layers"][2]["weights_of"] = 1                 # two layers that lead to one another
    at = cfg
    for key in path[:-1]:
        at = at[key]
    if value is None:
        at.pop(path[-1])
    else:
        at[path[-1]] = value
    with pytest.raises(ConfigError) as error:
        KatadraConfig.from_dict(cfg)
    assert message in str(error.value)


@pytest.mark.parametrize("rows, reach", [(8, 30), (32, 600), (2, 50), (6, 40), (16, 16), (10, 5), (8, 64), (64, 256.5)])
def test_distance_table_against_the_formula(rows, reach):
    """Every distance up to past the reach: the table laid out once says what the formula says, and its
    last entry stands for all longer distances."""
    from mrun_b200.parts.gated_attention import distance_buckets
    table = distance_buckets(rows, reach)
    half = rows // 2
    assert table[:half] == list(range(half)) and table[-1] == rows - 1 and table == sorted(table)
    assert rows - 1 not in table[:-1]
    for n in range(half, int(2 * reach) + 40):
        if reach <= half:
            want = rows - 1
        else:
            want = plain.bucket(n, rows, reach)
        assert table[min(n, len(table) - 1)] == want, n


def test_hand_worked_values():
    # layer norm of (1, 3): mean 2, variance 1
    y = plain.layer_norm(torch.tensor([[1.0, 3.0]], dtype=F), torch.tensor([2.0, 5.0], dtype=F), torch.tensor([0.5, 0.0], dtype=F), 0.0)
    assert torch.allclose(y, torch.tensor([[-1.5, 5.0]], dtype=F))
    # buckets of a table of 8 rows that reaches 64: 4 * 16^(k / 4) begins bucket 4 + k
    assert [plain.bucket(n, 8, 64) for n in (0, 3, 4, 7, 8, 15, 16, 31, 32, 63, 64, 9999)] == [0, 3, 4, 4, 5, 5, 6, 6, 7, 7, 7, 7]
    # temperatures: 1 + ln 1 up to the block's last position, then 1 + coef ln 2
    t = plain.temperature(torch.tensor([0, 8, 9, 18, 19]), 0.5, 10)
    assert torch.allclose(t, torch.tensor([1, 1, 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(3)], dtype=F))
    assert abs(float(plain.soft_cap(torch.tensor(1e9, dtype=F), 7.0)) - 7.0) < 1e-9
    # the row before the first token is zero
    h = torch.tensor([[2.0], [6.0]], dtype=F)
    assert torch.allclose(plain.token_shift(h, torch.tensor([0.25], dtype=F)), torch.tensor([[1.5], [5.0]], dtype=F))
    # one channel: o_0 = u k_0 v_0 r_0, then S_0 = k_0 v_0, o_1 = (S_0 + u k_1 v_1) r_1, S_1 = w_1 S_0 + k_1 v_1
    col = lambda *x: torch.tensor(x, dtype=F).view(-1, 1, 1)
    o = plain.bonus_recurrence(col(1, 2, 1), col(3, 1, 0), col(5, 7, 0), col(0.5, 0.1, 0.2), torch.tensor([[0.5]], dtype=F))
    assert torch.allclose(o.flatten(), torch.tensor([7.5, 2 * (15 + 3.5), 0.1 * 15 + 7], dtype=F))
    # one channel of the state space: dt = (1, 2), e^a_log = ln 2: the state halves, then quarters
    y = plain.state_space(col(3, 5), col(1, 1), col(1, 10), torch.tensor([[1.0], [2.0]], dtype=F), torch.tensor([math.log(math.log(2))], dtype=F))
    assert torch.allclose(y.flatten(), torch.tensor([3.0, 10 * (3 / 4 + 10)], dtype=F))
    # a convolution of two taps with a bias: w0 x_(t-1) + w1 x_t + b, through SiLU
    x, w, b = torch.tensor([[1.0], [2.0]], dtype=F), torch.tensor([[10.0, 1.0]], dtype=F), torch.tensor([0.5], dtype=F)
    assert torch.allclose(plain.short_conv(x, w, b), plain.silu(torch.tensor([[1.5], [12.5]], dtype=F)))
    W = {"m.up": torch.tensor([[1.0], [-1.0]], dtype=F), "m.down": torch.tensor([[2.0, 3.0]], dtype=F)}
    assert torch.allclose(plain.dense_feed_forward(W, "m.", torch.tensor([[4.0], [-2.0]], dtype=F)), torch.tensor([[32.0], [12.0]], dtype=F))


def test_shared_layers_run_their_owner_again(tmp_path):
    """A model whose third layer runs the first one's weights is the model in which they are written twice."""
    cfg, weights = load_folder(make_folder("mixed", str(tmp_path / "m")))
    written = copy.deepcopy(cfg)
    written["layers"][2].pop("weights_of")
    both = dict(weights, **{n.replace("l0.", "l2.", 1): t for n, t in weights.items() if n.startswith("l0.")})
    tokens = list(range(20))
    assert torch.equal(plain.forward(cfg, weights, tokens), plain.forward(written, both, tokens))


def test_two_mixers_side_by_side_need_names_of_their_own():
    from mrun_b200.cache.needs import FixedState, PagedKV, split_need
    from mrun_b200.parts import MIXERS, Precision, Runtime
    spec = kconfig("odd").to_spec().layers[1].mixer
    rt = Runtime(torch.device("cpu"), Precision.of("float32"), 8)
    w = {t.name[2:]: torch.zeros(t.shape) for t in MIXERS.tensor_specs(spec, "m")}
    part = MIXERS.build(spec, w, rt)
    paged, states = split_need(part.cache_need())
    assert paged == PagedKV(1, 11, None, value_dim=5)
    assert {s.name: s for s in states} == {"state": FixedState((3, 13, 13), "float32", "state"),
                                           "shift": FixedState((1, 37), "float32", "shift")}
    assert part.w_o.shape == (37, 3 * 5 + 3 * 13) and part.graph_safe
