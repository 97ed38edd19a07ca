"""Fusanex on the host: the configuration's checks, the plan, the cache groups and state that follow from it, and the plain
statement's own pieces."""
import copy
import math

import pytest
import torch

import plain_fusanex as plain
from fusanex_configs import CONFIGS, shaped_weights, write_tensors


def typed(raw):
    from wllm_b200.config import FusanexConfig
    return FusanexConfig.from_dict(raw, where="test")


def model_of(raw, dtype=torch.bfloat16):
    from wllm_b200.config import resolve_architecture
    from wllm_b200.engine.model import ComposedModel
    return ComposedModel(resolve_architecture("Fusanex").make_plan(typed(raw)), dtype)


@pytest.mark.parametrize("name", list(CONFIGS))
def test_round_trip_and_defaults(name):
    cfg = typed(CONFIGS[name])
    assert typed(cfg.to_dict()) == cfg
    assert cfg.norm_groups == CONFIGS[name]["norm"].get("groups", 1)
    assert cfg.embedding_scale == (CONFIGS[name].get("embedding") or {}).get("scale", 1.0)
    for layer, raw in zip(cfg.layers, CONFIGS[name]["layers"]):
        if layer["type"] == "parallel":
            left, rl = layer["mixer"]["left"], raw["mixer"]["left"]
            assert left["kv_heads"] == rl.get("kv_heads", rl["heads"]) and left["vdim"] == rl.get("vdim", rl["dim"])
            assert left["scale"] == rl.get("scale", rl["dim"] ** -0.5) and ("q_temp" in left) == ("q_temp" in rl)
            assert layer["mixer"]["left_scale"] == raw["mixer"].get("left_scale", 1.0)
        if layer["mlp"] is not None:
            assert layer["mlp"]["router"]["identity"] == raw["mlp"]["router"].get("identity", 0)
            assert ("shared" in layer["mlp"]) == ("shared" in raw["mlp"])


def test_every_problem_is_named_at_once():
    from wllm_b200.config import ConfigError
    raw = copy.deepcopy(CONFIGS["mixed"])
    del raw["vocab"]
    raw["norm"]["groups"] = 7
    raw["layers"][0]["mixer"]["blocks"] = 5
    raw["layers"][0]["mlp"]["router"]["top"] = 9
    raw["layers"][1]["mixer"]["left"]["kv_heads"] = 3
    raw["layers"][1]["mixer"]["left"]["q_temp"]["every"] = 0
    raw["layers"][2]["type"] = "conv"
    raw["layers"][3]["mlp"]["kind"] = "dense"
    del raw["layers"][4]["mlp"]["expert"]["limit"]
    with pytest.raises(ConfigError) as e:
        typed(raw)
    text = str(e.value)
    for piece in ("vocab", "64 is no multiple of 7", "48 is no multiple of 5", "top 9 of 8", "4 heads are no multiple of 3", "every", "layers[2].type",
                  "layers[3].mlp.kind", "limit"):
        assert piece in text, (piece, text)


def test_the_plan_names_every_tensor_and_no_other():
    model = model_of(CONFIGS["mixed"])
    names = {ps.name: ps.shape for ps in model.param_specs()}
    assert {"embed", "final.norm", "head"} <= set(names)
    assert names["l0.mix.y"] == (48, 64) and names["l0.mix.conv"] == (48, 4) and names["l0.mix.ra"] == (3, 16, 16) and names["l0.mix.ri.b"] == (3, 16)
    assert names["l1.mix.left.q.norm"] == (16,) and names["l1.mix.left.v"] == (48, 64) and names["l1.mix.left.o"] == (64, 96)
    assert names["l1.mix.right.mu.w"] == (64,) and names["l1.mix.right.w1"] == (12, 64) and names["l1.mix.right.w2"] == (48, 12)
    assert names["l1.mix.right.u"] == (2, 24) and names["l1.mix.right.norm"] == (48,)
    assert names["l0.mlp.router"] == (8, 64) == (names["l0.mlp.correction"][0], 64) and "l0.mlp.e6.up" not in names and "l0.mlp.e5.up" in names
    assert names["l0.mlp.shared.down"] == (64, 24) and "l4.mlp.shared.up" not in names
    assert "l2.norm2" not in names and "l2.mlp.router" not in names


def test_cache_groups_and_state_follow_from_the_mixers():
    model = model_of(CONFIGS["mixed"])
    assert {g.name for g in model.group_specs} == {"all-2x16v24", "all-2x16"}
    states = {s.name: (tuple(s.shape), s.dtype) for s in model.state_specs}
    assert states["run0.state"] == ((48,), torch.float32) and states["run0.conv"] == ((4, 48), torch.float32)
    assert states["run1.right.state"] == ((2, 24, 24), torch.float32) and states["run1.right.row"] == ((2, 64), torch.bfloat16)
    assert states["run2.conv"] == ((3, 64), torch.float32) and len(states) == 10
    assert model.graph_safe


def test_a_rank_that_only_the_checkpoint_knows(tmp_path):
    """Without `rank` in the file the low-rank map's size comes from the tensors."""
    from wllm_b200.engine.model import ComposedModel
    from wllm_b200.config import config_from_folder
    from wllm_b200.weights import load_weights
    from wllm_b200.weights.loader import WeightError
    raw = copy.deepcopy(CONFIGS["bare"])
    tensors = shaped_weights(raw, 5)
    for layer in raw["layers"]:
        layer["mixer"].get("right", {}).pop("rank", None)
    folder = write_tensors(str(tmp_path / "m"), raw, tensors)
    arch, cfg = config_from_folder(folder)
    model = ComposedModel(arch.make_plan(cfg), torch.float32)
    load_weights(model, folder, "cpu")
    assert [b.mixer.right.rank for b in model.blocks if hasattr(b.mixer, "right")] == [4, 8]
    tensors["l0.mix.right.w2"] = torch.zeros(16, 5)
    folder = write_tensors(str(tmp_path / "n"), raw, tensors)
    with pytest.raises((ValueError, WeightError)):
        load_weights(ComposedModel(arch.make_plan(cfg), torch.float32), folder, "cpu")


def test_a_factor_of_zero_leaves_the_other_side(tmp_path):
    from wllm_b200.engine.model import ComposedModel
    from wllm_b200.config import config_from_folder
    from wllm_b200.weights import load_weights
    raw = copy.deepcopy(CONFIGS["bare"])
    raw["layers"][0]["mixer"].update(left_scale=0.0, right_scale=0.3)
    folder = write_tensors(str(tmp_path / "m"), raw, shaped_weights(raw, 5))
    arch, cfg = config_from_folder(folder)
    model = ComposedModel(arch.make_plan(cfg), torch.float32)
    load_weights(model, folder, "cpu")
    m = model.blocks[0].mixer
    assert m.factor == 0.3 and m.ratio == 1.0 and float(m.w_out[:, :m.left_out].abs().max()) == 0.0
    assert float(m.w_out[:, m.left_out:m.left_out + m.right.out_width].abs().max()) > 0.0


def test_the_plain_statements_pieces():
    x = torch.arange(1.0, 6.0)[:, None]
    taps = torch.tensor([[100.0, 10.0, 1.0]])
    assert plain.short_conv(x, taps, torch.tensor([0.5]))[:, 0].tolist() == [1.5, 12.5, 123.5, 234.5, 345.5]     # the last tap is the token's own
    # the norm's groups do not see one another
    y = plain.group_norm(torch.tensor([[3.0, 4.0, 300.0, 400.0]], dtype=torch.float64), torch.ones(4, dtype=torch.float64), 2, 0.0)
    assert torch.allclose(y[0, :2], y[0, 2:]) and torch.allclose(y[0, :2], torch.tensor([3.0, 4.0], dtype=torch.float64) / math.sqrt(12.5))
    t = plain.temperature(torch.arange(6), 3, 0.5, torch.float64)
    assert t[:2].tolist() == [1.0, 1.0] and torch.allclose(t[2:5], torch.full((3,), 1 + 0.5 * math.log(2), dtype=torch.float64)) and t[5] > t[4]
    # the first token's state has nothing to decay; an input is kept sqrt(1 - a^2) times
    r, lam = torch.full((2, 1), 0.5, dtype=torch.float64), torch.zeros(1, dtype=torch.float64)
    a = math.exp(-4.0 * math.log(2.0))
    S = plain.lru(torch.ones(2, 1, dtype=torch.float64), r, torch.ones(2, 1, dtype=torch.float64), lam)
    assert math.isclose(float(S[0]), math.sqrt(1 - a * a)) and math.isclose(float(S[1]), (1 + a) * math.sqrt(1 - a * a))
    # the bonus counts the token's own key and value, and no other's
    one = torch.ones(3, 1, 1, dtype=torch.float64)
    o = plain.time_mix(one, one, one * torch.tensor([1.0, 10.0, 100.0], dtype=torch.float64)[:, None, None], one * 0.5, torch.full((1, 1), 7.0, dtype=torch.float64))
    assert o[:, 0, 0].tolist() == [7.0, 71.0, 710.5]
    # the correction chooses, the weights do not see it; an identity expert gives the row back
    h = torch.tensor([[1.0, 2.0]], dtype=torch.float64)
    w = {"router": torch.zeros(3, 2, dtype=torch.float64), "correction": torch.tensor([0.0, 0.1, 0.2], dtype=torch.float64),
         "e0.gate": torch.zeros(1, 2, dtype=torch.float64), "e0.up": torch.zeros(1, 2, dtype=torch.float64), "e0.down": torch.zeros(2, 1, dtype=torch.float64)}
    w.update({k.replace("e0", "e1"): v for k, v in w.items() if k.startswith("e0")})
    mlp = {"router": {"experts": 2, "top": 2, "identity": 1}, "expert": {"ff": 1, "limit": 1.0}}
    idx, val = plain.route(mlp, w, "", h)
    assert idx[0].tolist() == [2, 1] and torch.allclose(val, torch.full((1, 2), 0.5, dtype=torch.float64))
    assert torch.allclose(plain.experts_ff(mlp, w, "", h), 0.5 * h)
