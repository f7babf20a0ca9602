"""Katopel without a GPU: the configuration and its errors, the plan's tensors and run list, cache requests, shared rotation tables,
tensors that a layer without feed-forward may carry, and the plain implementation's own mechanisms on cases small enough to work
out by hand."""

import copy
import json
import math

import pytest
import torch

from tests.katopel_configs import KAT_A, KAT_B, KAT_C, KAT_CONFIGS, KAT_D
from tests.plain import katopel as plain


def _model(raw, dtype=torch.float32):
    from gtar_kimik3_public_b200.models.model import Model
    from gtar_kimik3_public_b200.registry import architecture, config_from_dict

    config = config_from_dict(raw)
    return Model(architecture("Katopel").build_plan(config), config, dtype, "cpu")


def _delta_tensors(p, m, W):
    H, G, d, dv, taps = (m[k] for k in ("heads", "kv_heads", "dim", "vdim", "conv"))
    out = {p + n: (size, W) for n, size in (("q", G * d), ("k", G * d), ("v", H * dv), ("b", H), ("a", H), ("g", H * dv))}
    out.update({p + n + ".conv": (size, taps) for n, size in (("q", G * d), ("k", G * d), ("v", H * dv))})
    return {**out, p + "A_log": (H,), p + "dt_bias": (H,), p + "norm": (dv,), p + "o": (W, H * dv)}


@pytest.mark.parametrize("tag", sorted(KAT_CONFIGS))
def test_configurations_are_read_and_give_their_tensors(tag):
    raw = KAT_CONFIGS[tag]
    W = raw["width"]
    model = _model(raw)
    specs = {name: spec.shape for name, spec in model.tensor_specs().items() if not spec.optional}
    want = {"embed": (raw["vocab"], W), "final.norm": (W,), "final.norm.b": (W,)}
    if "loop" in raw:
        want["loop.step"] = (raw["loop"]["times"], W)
    for i, layer in enumerate(raw["layers"]):
        m, mlp, p = layer["mixer"], layer["mlp"], f"l{i}.mix."
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if mlp is not None else ()):
            want.update({f"l{i}.{n}": (W,), f"l{i}.{n}.b": (W,)})
        if layer["type"] == "delta":
            want.update(_delta_tensors(p, m, W))
        else:
            want.update(_delta_tensors(p + "right.", m["right"], W))
            a = m["left"]
            for n, size in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                want.update({p + "left." + n: (size, W), p + "left." + n + ".b": (size,)})
            want[p + "left.o"] = (W, a["heads"] * a["vdim"])
        p = f"l{i}.mlp."
        if mlp is None:
            continue
        feed = [("", mlp["ff"])] if mlp["kind"] == "dense" else [(f"e{e}.", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
        if "shared" in mlp:
            feed.append(("shared.", mlp["shared"]["ff"]))
            want[p + "shared.sg"] = (1, W)
        if mlp["kind"] == "moe":
            want[p + "router"] = (mlp["router"]["experts"], W)
        for name, ff in feed:
            want.update({p + name + "gate": (ff, W), p + name + "up": (ff, W), p + name + "down": (W, ff)})
    assert specs == want
    assert model.graph_safe()


def test_run_lists():
    from gtar_kimik3_public_b200.models.model import Enter, looped_run_list

    runs = [(e.layer, e.enter, e.cache_of) for e in _model(KAT_A).plan.run_list]
    first, again, third = Enter(False, 0), Enter(True, 1), Enter(True, 2)
    assert runs == [(0, None, None), (1, first, None), (2, None, None), (1, again, None), (2, None, None), (1, third, None), (2, None, None),
                    (3, None, None)]
    assert [(e.layer, e.enter) for e in _model(KAT_C).plan.run_list] == [(0, None), (1, None), (2, first), (2, again)]
    assert [(e.layer, e.enter) for e in _model(KAT_D).plan.run_list] == [(0, None), (1, first), (2, None), (3, None)]
    raw = copy.deepcopy(KAT_A)
    del raw["loop"]
    plan = _model(raw).plan
    assert [(e.layer, e.enter) for e in plan.run_list] == [(i, None) for i in range(4)] and plan.steps is None
    assert [(e.layer, e.enter) for e in looped_run_list(2, 0, 1, 2)] == [(0, None), (0, Enter(True, None)), (1, None)]
    for bad in ((2, 1, 1, 2), (2, 0, 3, 1), (2, 0, 1, 0)):
        with pytest.raises(ValueError):
            looped_run_list(*bad)
    # the plain implementation's own order of execution
    for tag, raw in KAT_CONFIGS.items():
        ours = [(e.layer, None if e.enter is None else e.enter.step) for e in _model(raw).plan.run_list]
        assert ours == plain.run_order(raw), tag


def test_every_pass_has_a_cache_of_its_own():
    from gtar_kimik3_public_b200.parts.base import KVRequest, StateRequest

    requests = _model(KAT_A).cache_layout().requests
    pair = [KVRequest(2, 16, 17, value_dim=24), StateRequest((3, 16, 32), torch.float32), StateRequest((4, 2 * 16 + 3 * 32), torch.float32)]
    assert requests[1] == requests[3] == requests[5] == pair and len(requests) == 8
    assert requests[0] == [StateRequest((4, 24, 40), torch.float32), StateRequest((3, 2 * 2 * 24 + 4 * 40), torch.float32)]
    # no chunks: every key stays; a convolution of one tap keeps nothing; values as wide as keys
    assert _model(KAT_B).cache_layout().requests[2][0] == KVRequest(1, 128, None)
    assert _model(KAT_C).cache_layout().requests[2] == [StateRequest((3, 64, 96), torch.float32)]
    model = _model(KAT_A, torch.bfloat16)
    cache = model.make_cache(256, 2)
    passes = [cache.view(i) for i in (1, 3, 5)]
    assert len({v[1].data_ptr() for v in passes}) == 3 and len({v[0].k.data_ptr() for v in passes}) == 3


def test_layers_with_equal_rotations_share_a_table():
    raw = copy.deepcopy(KAT_A)
    raw["layers"].append(copy.deepcopy(raw["layers"][1]))
    raw["layers"].append(copy.deepcopy(raw["layers"][1]))
    raw["layers"][5]["mixer"]["left"]["rot"]["base"] = 77.0
    plan = _model(raw).plan
    assert len(plan.positions) == 3
    position = lambda i: plan.layers[i].mixer.left.position
    assert position(1) is position(4) is not position(5) and _model(KAT_D).plan.layers[2].mixer.left.position is None


def test_a_layer_without_feed_forward_may_carry_the_absent_branchs_norms(tmp_path):
    from gtar_kimik3_public_b200.weights.loader import WeightsError, check_tensors

    specs = _model(KAT_D).tensor_specs()
    have = {name: tuple(spec.shape) for name, spec in specs.items() if not spec.optional}
    assert "l0.norm2" not in have and "l1.norm2b.b" in have
    check_tensors(tmp_path, specs, have, {})
    check_tensors(tmp_path, specs, {**have, "l0.norm2": (42,), "l0.norm2.b": (42,), "l0.norm2b": (42,), "l0.norm2b.b": (42,)}, {})
    for extra in ("l0.norm3", "l0.mlp.up", "l1.mix.q", "loop.scale"):
        with pytest.raises(WeightsError):
            check_tensors(tmp_path, specs, {**have, extra: (4,)}, {})
    with pytest.raises(WeightsError):
        check_tensors(tmp_path, specs, {k: v for k, v in have.items() if k != "loop.step"}, {})


def _changed(path, value):
    raw = copy.deepcopy(KAT_A)
    at = raw
    for key in path[:-1]:
        at = at[key]
    if value is KeyError:
        del at[path[-1]]
    else:
        at[path[-1]] = value
    return raw


@pytest.mark.parametrize("change,message", [
    ((("layers", 0, "type"), "mamba"), "not a mixer"),
    ((("layers", 0, "mixer", "conv"), KeyError), "missing keys ['conv']"),
    ((("layers", 0, "mixer", "conv"), 17), "conv must be at most 16"),
    ((("layers", 0, "mixer", "dim"), 513), "dim must be at most 512"),
    ((("layers", 0, "mixer", "heads"), 3), "multiple of kv_heads"),
    ((("layers", 0, "mixer", "decay"), 1.0), "unknown keys ['decay']"),
    ((("layers", 1, "mixer", "middle"), {}), "unknown keys ['middle']"),
    ((("layers", 1, "mixer", "right"), KeyError), "missing keys ['right']"),
    ((("layers", 1, "mixer", "left", "rot", "dims"), 5), "rot.dims"),
    ((("layers", 1, "mixer", "left", "rot", "dims"), 18), "rot.dims"),
    ((("layers", 1, "mixer", "left", "scale"), 0), "scale"),
    ((("layers", 1, "mixer", "left", "mask"), {}), "missing keys ['size']"),
    ((("layers", 1, "mixer", "left", "mask", "size"), 2.5), "mask.size"),
    ((("layers", 1, "mixer", "left_scale"), "big"), "left_scale"),
    ((("layers", 1, "mlp", "kind"), "swiglu"), "mlp.kind"),
    ((("layers", 1, "mlp", "router", "top"), 7), "cannot be chosen"),
    ((("layers", 1, "mlp", "router", "groups"), {}), "unknown keys ['groups']"),
    ((("layers", 1, "mlp", "shared"), {}), "missing keys ['ff']"),
    ((("loop", "stop"), 5), "are not layers"),
    ((("loop", "stop"), 1), "are not layers"),
    ((("loop", "times"), 0), "loop.times"),
    ((("loop", "start"), -1), "loop.start"),
    ((("norm",), {}), "missing keys ['eps']"),
    ((("depth",), 3), "unknown keys ['depth']"),
])
def test_configuration_errors_name_the_key(change, message):
    from gtar_kimik3_public_b200.config.base import ConfigError
    from gtar_kimik3_public_b200.registry import config_from_dict

    with pytest.raises(ConfigError) as caught:
        config_from_dict(_changed(*change))
    assert message in str(caught.value)


def test_a_configuration_survives_its_own_file(tmp_path):
    from gtar_kimik3_public_b200.registry import config_from_dict, config_from_file

    config = config_from_dict(KAT_C)
    (tmp_path / "config.json").write_text(json.dumps(config.to_dict()))
    again = config_from_file(tmp_path)
    assert again == config and again.embedding_scale == 0.5 and config_from_dict(KAT_B).embedding_scale == 1.0


def test_logits_come_from_the_embedding_table_without_its_constant():
    model = _model(KAT_A)
    tensors = {name: torch.randn(spec.shape) for name, spec in model.tensor_specs().items() if not spec.optional}
    model.load(tensors)
    assert model.plan.head.weight is model.plan.embedding.weight and torch.equal(model.plan.head.weight, tensors["embed"])
    assert model.plan.embedding.scale == 3.0 and model.plan.head.scale == 1.0


def test_a_pair_of_mixers_is_packed_into_two_products():
    model = _model(KAT_A)
    tensors = {name: torch.randn(spec.shape) for name, spec in model.tensor_specs().items() if not spec.optional}
    model.load(tensors)
    pair = model.plan.layers[1].mixer
    assert pair.left.w_in is None and pair.right.w_in is None and pair.right_at % 8 == 0
    assert torch.equal(pair.w_in[:96], tensors["l1.mix.left.q"])
    assert torch.equal(pair.w_in[pair.right_at:pair.right_at + 16], tensors["l1.mix.right.q"])
    assert torch.equal(pair.w_o, torch.cat([tensors["l1.mix.left.o"], tensors["l1.mix.right.o"]], dim=1))
    assert pair.weight_bytes() >= 4 * (pair.w_in.numel() + pair.w_o.numel())


# ------------------------------------------------------------------ the plain implementation by hand
def test_plain_delta_rule_by_hand():
    one = torch.ones(2, 1, dtype=torch.float64)
    q, k = one * 2.0, torch.tensor([[0.5], [3.0]], dtype=torch.float64)
    v, g, beta = torch.tensor([[5.0], [7.0]], dtype=torch.float64), torch.tensor([0.9, 0.25]), torch.tensor([0.5, 0.75])
    got = plain.delta_scan(q, k, v, g, beta)
    s0 = 0.5 * 0.5 * 5.0
    assert math.isclose(got[0, 0].item(), 2.0 * s0, rel_tol=1e-12)  # the read-out sees its own token's write
    faded = 0.25 * s0
    s1 = faded + 3.0 * 0.75 * (7.0 - 3.0 * faded)  # the decay comes before the correction
    assert math.isclose(got[1, 0].item(), 2.0 * s1, rel_tol=1e-12)


def test_plain_convolution_by_hand():
    x = torch.tensor([[1.0], [10.0], [100.0]], dtype=torch.float64)
    got = plain.over_time(x, torch.tensor([[3.0, 2.0, 1.0]], dtype=torch.float64))[:, 0].tolist()
    assert got == [1.0, 12.0, 123.0]  # the last tap is the current token's
    assert plain.over_time(x[:1], torch.ones(1, 5, dtype=torch.float64)).tolist() == [[1.0]]


def test_plain_chunks_by_hand():
    seen = plain.same_chunk(7, 3)
    assert seen[5].tolist() == [False, False, False, True, True, True, False]
    assert seen[6].tolist() == [False] * 6 + [True] and seen[2].tolist() == [True] * 3 + [False] * 4
    assert plain.same_chunk(4, None)[3].sum() == 4


def test_plain_layer_norm_by_hand():
    w = {"n": torch.tensor([2.0, 1.0], dtype=torch.float64), "n.b": torch.tensor([0.5, -1.0], dtype=torch.float64)}
    got = plain.layer_norm(torch.tensor([[1.0, 5.0]], dtype=torch.float64), w, "n", 0.25)
    r = math.sqrt(4.0 + 0.25)
    assert torch.allclose(got, torch.tensor([[2.0 * -2.0 / r + 0.5, 2.0 / r - 1.0]], dtype=torch.float64))


def test_plain_rotation_turns_neighbours_of_part_of_a_head():
    x = torch.randn(6, 2, 8, dtype=torch.float64, generator=torch.Generator().manual_seed(1))
    got = plain.turn_pairs(x, 9.0, 4)
    a = 5 * 9.0 ** (-2.0 / 4)  # position 5, the second pair: entries 2 and 3; the exponent counts the rotated entries
    assert math.isclose(got[5, 1, 2].item(), x[5, 1, 2].item() * math.cos(a) - x[5, 1, 3].item() * math.sin(a), abs_tol=1e-12)
    assert math.isclose(got[5, 1, 3].item(), x[5, 1, 3].item() * math.cos(a) + x[5, 1, 2].item() * math.sin(a), abs_tol=1e-12)
    assert torch.equal(got[..., 4:], x[..., 4:]) and torch.equal(got[0], x[0])


def test_plain_router_by_hand():
    h = torch.eye(2, dtype=torch.float64)
    w = {"r.router": torch.tensor([[1.0, 0.0], [2.0, 0.0], [0.0, 3.0]], dtype=torch.float64)}
    ids, share = plain.route(h, w, "r.", {"experts": 3, "top": 2})
    assert ids[0].tolist() == [1, 0]
    assert math.isclose(share[0, 0].item(), math.e ** 2 / (math.e ** 2 + math.e), rel_tol=1e-12)  # over the chosen alone
