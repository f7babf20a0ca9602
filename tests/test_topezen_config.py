"""Topezen without a GPU: the configuration and its errors, the plan's tensors, cache requests, shared rotation tables, the
order of rotated entries that the latent attention sets at load, norms of one number, the random-weights mode, and the plain
implementation's own mechanisms on cases small enough to work out by hand."""

import copy
import json
import math

import pytest
import torch

from tests.plain import topezen as plain
from tests.topezen_configs import TPZ_A, TPZ_B, TPZ_C, TPZ_CONFIGS, TPZ_D


def _model(raw, dtype=torch.float32):
    from gtar_kimik3_public_b200.models.model import Model
    from gtar_kimik3_public_b200.registry import architecture, config_from_dict

    config = config_from_dict(raw)
    return Model(architecture("Topezen").build_plan(config), config, dtype, "cpu")


@pytest.mark.parametrize("tag", sorted(TPZ_CONFIGS))
def test_configurations_are_read_and_give_their_tensors(tag):
    raw = TPZ_CONFIGS[tag]
    W = raw["width"]
    model = _model(raw)
    specs = {name: spec.shape for name, spec in model.tensor_specs().items() if not spec.optional}
    want = {"embed": (raw["vocab"], W), "head": (raw["vocab"], W), "final.norm": ()}
    for i, layer in enumerate(raw["layers"]):
        m, mlp = layer["mixer"], layer["mlp"]
        p = f"l{i}.mix."
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        for n in (1, 2) if mlp is not None else (1,):
            want.update({f"l{i}.norm{n}": (), f"l{i}.rg{n}": (W, W), f"l{i}.rg{n}.b": (W,)})
        want[p + "o"] = (W, H * dv)
        if layer["type"] == "mlstm":
            want.update({p + "q": (H * d, W), p + "k": (H * d, W), p + "v": (H * dv, W), p + "g": (H * dv, W), p + "i": (H, W), p + "i.b": (H,),
                         p + "f": (H, W), p + "f.b": (H,), p + "norm": (H * dv,)})
        elif layer["type"] == "attention":
            G = m["kv_heads"]
            want.update({p + "q": (H * d, W), p + "k": (G * d, W), p + "v": (G * dv, W), p + "q.norm": (d,), p + "k.norm": (d,), p + "sink": (H,)})
        else:
            r, qr, kr = m["rot_dim"], m["q_rank"], m["kv_rank"]
            want.update({p + "dq": (qr, W), p + "dq.norm": (qr,), p + "uq": (H * (d + r), qr), p + "dkv": (kr + r, W), p + "dkv.norm": (kr,),
                         p + "uk": (H * d, kr), p + "uv": (H * dv, kr), p + "g": (H * dv, W)})
        p = f"l{i}.mlp."
        if mlp is not None and mlp["kind"] == "dense":
            want.update({p + "up": (mlp["ff"], W), p + "down": (W, mlp["ff"]), p + "act": (4,)})
        elif mlp is not None:
            experts = [(f"e{e}.", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
            experts += [("shared.", mlp["shared"]["ff"])] if "shared" in mlp else []
            for name, ff in experts:
                want.update({p + name + "gate": (ff, W), p + name + "up": (ff, W), p + name + "down": (W, ff)})
            want.update({p + "router": (mlp["router"]["experts"], W), p + "correction": (mlp["router"]["experts"],)})
    assert specs == want
    assert model.graph_safe()


def test_a_layer_without_feed_forward_may_carry_the_absent_branchs_tensors(tmp_path):
    """A file whose layer has no feed-forward loads with and without the second norm and gate; other names are refused."""
    from gtar_kimik3_public_b200.weights.loader import WeightsError, check_tensors

    specs = _model(TPZ_D).tensor_specs()
    have = {name: tuple(spec.shape) for name, spec in specs.items() if not spec.optional}
    assert "l0.rg2" not in have and "l1.rg2" in have
    check_tensors(tmp_path, specs, have, {})
    check_tensors(tmp_path, specs, {**have, "l0.norm2": (), "l0.rg2": (42, 42), "l0.rg2.b": (42,)}, {})
    for extra in ("l0.norm3", "l0.mlp.up", "l1.mlp.shared.up"):
        with pytest.raises(WeightsError):
            check_tensors(tmp_path, specs, {**have, extra: (4,)}, {})


def test_cache_requests():
    from gtar_kimik3_public_b200.parts.base import KVRequest, RowsRequest, StateRequest

    requests = _model(TPZ_A).cache_layout().requests
    assert requests[0] == RowsRequest(24 + 12, None)
    assert requests[1] == [StateRequest((3, 25, 40), torch.float32), StateRequest((3, 25), torch.float32)]
    assert requests[2] == KVRequest(2, 16, 17, value_dim=24, keep_first=3)
    assert requests[4] == KVRequest(4, 24, None)
    # no kept first tokens, one kept, more kept than the window is long
    requests = _model(TPZ_D).cache_layout().requests
    assert requests[1] == KVRequest(1, 10, 1, value_dim=14, keep_first=1) and requests[3] == KVRequest(2, 6, 200, keep_first=0)
    assert _model(TPZ_C).cache_layout().requests[0] == KVRequest(1, 128, 65, keep_first=130)


def test_layers_with_equal_rotations_share_a_table():
    raw = copy.deepcopy(TPZ_B)
    raw["layers"].append(copy.deepcopy(raw["layers"][2]))
    raw["layers"].append(copy.deepcopy(raw["layers"][2]))
    raw["layers"][5]["mixer"]["rot"]["base"] = 77.0
    plan = _model(raw).plan
    assert len(plan.positions) == 2
    assert plan.layers[2].mixer.position is plan.layers[4].mixer.position is not plan.layers[5].mixer.position


def _changed(path, value):
    raw = copy.deepcopy(TPZ_A)
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
    ((("layers", 0, "mixer", "rot"), KeyError), "missing keys ['rot']"),
    ((("layers", 0, "mixer", "rot", "dims"), 10), "rot.dims"),
    ((("layers", 0, "mixer", "window"), 4), "unknown keys ['window']"),
    ((("layers", 0, "mixer", "q_rank"), 0), "q_rank"),
    ((("layers", 1, "mixer", "gate_cap"), 0), "gate_cap"),
    ((("layers", 1, "mixer", "gate_cap"), KeyError), "missing keys ['gate_cap']"),
    ((("layers", 2, "mixer", "heads"), 5), "multiple of kv_heads"),
    ((("layers", 2, "mixer", "softcap"), -1.0), "softcap"),
    ((("layers", 2, "mixer", "mask"), {"keep_first": 4}), "missing keys ['size']"),
    ((("layers", 2, "mixer", "mask", "keep_first"), -1), "keep_first"),
    ((("layers", 2, "mixer", "mask", "size"), 2.5), "mask.size"),
    ((("layers", 1, "mlp", "kind"), "swiglu"), "mlp.kind"),
    ((("layers", 0, "mlp", "router", "top"), 5), "cannot be chosen"),
    ((("layers", 0, "mlp", "router", "groups", "count"), 4), "equal groups"),
    ((("layers", 0, "mlp", "router", "groups", "keep"), 4), "equal groups"),
    ((("layers", 0, "mlp", "shared"), {}), "missing keys ['ff']"),
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

    config = config_from_dict(TPZ_C)
    (tmp_path / "config.json").write_text(json.dumps(config.to_dict()))
    again = config_from_file(tmp_path)
    assert again == config and again.embedding_scale == 0.5 and config_from_dict(TPZ_B).embedding_scale == 1.0


def test_numbers_without_dimensions_travel_through_the_file(tmp_path):
    """A norm's one number is a tensor without dimensions: written, checked and read back as such."""
    from gtar_kimik3_public_b200.registry import config_from_dict
    from gtar_kimik3_public_b200.weights import write_random_model
    from gtar_kimik3_public_b200.weights.safetensors_io import ModelFolderTensors
    from tests.plain.weights import read_safetensors

    write_random_model(tmp_path, config_from_dict(TPZ_D), seed=3, std=0.1)
    theirs = read_safetensors(tmp_path / "model.safetensors")
    ours = ModelFolderTensors(tmp_path)
    assert theirs["l0.norm1"].shape == () == tuple(ours.shape("final.norm"))
    model = _model(TPZ_D)
    model.load({name: ours.tensor(name).float() for name in ours.names()})
    block = model.plan.layers[1]
    assert block.norm_1.gain == pytest.approx(theirs["l1.norm1"].item()) and block.norm_1.gain != block.norm_2.gain
    assert torch.equal(model.plan.final_norm.weight, theirs["final.norm"].float().expand(42))


def test_rotated_rows_are_put_in_the_order_of_the_kernels():
    """Neighbours that turn together stand half a part away from each other after loading: rotating those halves gives the
    plain rotation's numbers in the other order, for the queries' rows of every head and for the keys' rows alike."""
    from gtar_kimik3_public_b200.parts.base import build_part

    H, d, r, rank, W = 2, 5, 8, 6, 10
    position = build_part("position", "rope", dim=r, base=50.0, precise=True)
    part = build_part("mixer", "latent_attention", hidden_size=W, n_heads=H, head_dim=d, rot_dim=r, value_dim=4, q_rank=7, kv_rank=rank,
                      scale=1.0, norm_eps=1e-6, position=position, pairing="neighbours", gated=True)
    gen = torch.Generator().manual_seed(5)
    tensors = {name: torch.randn(spec.shape, generator=gen) for name, spec in part.tensor_specs().items()}
    part.load(tensors)
    order = [0, 2, 4, 6, 1, 3, 5, 7]
    uq, loaded = tensors["uq"].view(H, d + r, 7), part.w_uq.view(H, d + r, 7)
    assert torch.equal(loaded[:, :d], uq[:, :d]) and torch.equal(loaded[:, d:], uq[:, d:][:, order])
    assert torch.equal(part.w_down[7 + rank:7 + rank + r], tensors["dkv"][rank:][order])
    assert torch.equal(part.w_down[part.gate_at:part.gate_at + H * 4], tensors["g"])
    x = torch.randn(9, 1, r, generator=gen)
    turned = plain.turn_pairs(x, 50.0)
    position.prepare(9, torch.device("cpu"))
    cos, sin = position.cos[:9, None], position.sin[:9, None]
    u, v = x[..., order][..., :4], x[..., order][..., 4:]
    assert torch.allclose(torch.cat([u * cos - v * sin, v * cos + u * sin], -1), turned[..., order], atol=1e-5)


# ------------------------------------------------------------------ the plain implementation by hand
def test_plain_matrix_memory_by_hand():
    one = torch.ones(2, 1, dtype=torch.float64)
    q, k, v = one * 2.0, one * 3.0, torch.tensor([[5.0], [7.0]], dtype=torch.float64)
    i, f = torch.tensor([-4.0, 1.0], dtype=torch.float64), torch.tensor([-1.0, -0.5], dtype=torch.float64)
    got = plain.matrix_memory(q, k, v, i, f)
    # token 0: m = max(-1 + 0, -4) = -1 (a maximum that started at minus infinity would be -4)
    c0, n0 = math.exp(-4 + 1) * 15.0, math.exp(-4 + 1) * 3.0
    assert math.isclose(got[0, 0].item(), 2 * c0 / (max(2 * n0, math.exp(1.0)) + 1e-6), rel_tol=1e-12)
    # token 1: m = max(-0.5 - 1, 1) = 1
    c1, n1 = math.exp(-1.5 - 1) * c0 + 21.0, math.exp(-1.5 - 1) * n0 + 3.0
    assert math.isclose(got[1, 0].item(), 2 * c1 / (max(2 * n1, math.exp(-1.0)) + 1e-6), rel_tol=1e-12)


def test_plain_window_with_kept_first_tokens_by_hand():
    seen = plain.visible(7, {"size": 2, "keep_first": 2})
    assert seen[6].tolist() == [True, True, False, False, False, True, True]
    assert seen[1].tolist() == [True, True] + [False] * 5 and seen[0].sum() == 1
    assert plain.visible(5, {"size": 2})[4].tolist() == [False, False, False, True, True]
    assert plain.visible(5, None)[3].sum() == 4


def test_plain_polynorm_by_hand():
    z = torch.tensor([[1.0, -2.0]], dtype=torch.float64)
    got = plain.poly_norm(z, torch.tensor([0.5, 0.25, 2.0, -1.0], dtype=torch.float64), 1e-9)
    r1, r2, r3 = math.sqrt(2.5), math.sqrt(17 / 2), math.sqrt(65 / 2)
    want = [0.5 / r1 + 0.25 / r2 + 2 / r3 - 1, 0.5 * -2 / r1 + 0.25 * 4 / r2 + 2 * -8 / r3 - 1]
    assert torch.allclose(got, torch.tensor([want], dtype=torch.float64), atol=1e-8)


def test_plain_router_by_hand():
    h = torch.eye(2, dtype=torch.float64)
    z = torch.tensor([[1.0, 0.0], [2.0, 0.0], [0.0, 3.0], [1.5, 0.0]], dtype=torch.float64)
    w = {"r.router": z, "r.correction": torch.tensor([-1.0, -2.0, -1.2, -1.1], dtype=torch.float64)}
    ids, share = plain.route(h, w, "r.", {"experts": 4, "top": 2, "groups": {"count": 2, "keep": 1}})
    # token 0: scores ~ (e, e^2, 1, e^1.5) / sum; choice scores all negative; the second group's best (expert 3) is ahead
    s = torch.softmax(z[:, 0], -1)
    assert ids[0].tolist() == [3, 2] if (s[3] - 1.1) > (s[0] - 1.0) else [0, 1]
    chosen = s[ids[0]]
    assert torch.allclose(share[0], chosen / chosen.sum())


def test_plain_rotation_turns_neighbours():
    x = torch.randn(6, 2, 4, dtype=torch.float64, generator=torch.Generator().manual_seed(1))
    got = plain.turn_pairs(x, 9.0)
    a = 5 * 9.0 ** (-2.0 / 4)  # position 5, the second pair: entries 2 and 3
    assert math.isclose(got[5, 1, 2].item(), x[5, 1, 2].item() * math.cos(a) - x[5, 1, 3].item() * math.sin(a), abs_tol=1e-12)
    assert math.isclose(got[5, 1, 3].item(), x[5, 1, 3].item() * math.cos(a) + x[5, 1, 2].item() * math.sin(a), abs_tol=1e-12)
    assert torch.equal(got[0], x[0])
