"""Vifirax on the host: the configuration's checks, the plan, the cache groups and state that follow from it, the stretched
frequencies, and the plain statement's own pieces."""
import copy
import math

import pytest
import torch

import plain_vifirax as plain
from vifirax_configs import CONFIGS


def typed(raw):
    from wllm_b200.config import VifiraxConfig
    return VifiraxConfig.from_dict(raw, where="test")


def model_of(raw, dtype=torch.bfloat16):
    from wllm_b200.config import resolve_architecture
    from wllm_b200.engine.model import ComposedModel
    arch = resolve_architecture("Vifirax")
    return ComposedModel(arch.make_plan(typed(raw)), dtype)


@pytest.mark.parametrize("name", list(CONFIGS))
def test_round_trip_and_defaults(name):
    cfg = typed(CONFIGS[name])
    assert typed(cfg.to_dict()) == cfg
    assert cfg.logit_scale == CONFIGS[name].get("logit_scale", 1.0)
    for layer, raw in zip(cfg.layers, CONFIGS[name]["layers"]):
        m, r = layer["mixer"], raw["mixer"]
        if layer["type"] == "attention":
            assert m["vdim"] == r.get("vdim", m["dim"]) and m["scale"] == r.get("scale", m["dim"] ** -0.5) and m.get("rot") == r.get("rot")
        if layer["type"] == "mamba2":
            assert m["groups"] == r.get("groups", 1) and m["norm_groups"] == r.get("norm_groups", 1)


def test_every_problem_is_named_at_once():
    from wllm_b200.config import ConfigError
    raw = copy.deepcopy(CONFIGS["mixed"])
    del raw["vocab"]
    raw["layers"][0]["mixer"]["norm_groups"] = 7
    raw["layers"][1]["mixer"]["kv_heads"] = 3
    raw["layers"][2]["mixer"]["rot"]["dims"] = 40
    raw["layers"][3]["mixer"]["dim"] = 16              # its queries cannot meet layer 2's keys
    raw["layers"][3]["mlp"]["router"]["top"] = 9
    raw["layers"][4]["type"] = "conv"
    with pytest.raises(ConfigError) as e:
        typed(raw)
    for piece in ("vocab", "7 norm_groups", "4 heads are no multiple of 3", "dims 40", "cannot be read from layer 2", "top 9 of 5", "layers[4].type"):
        assert piece in str(e.value), (piece, str(e.value))
    for wrong in (4, 3, 0, 1):                         # a later layer, itself, a layer of another kind
        raw = copy.deepcopy(CONFIGS["mixed"])
        raw["layers"][3]["mixer"]["kv_from"] = wrong
        with pytest.raises(ConfigError, match="kv_from"):
            typed(raw)


def test_the_plan_names_every_tensor_and_no_other():
    names = {ps.name: tuple(ps.shape) for ps in model_of(CONFIGS["mixed"]).param_specs()}
    assert "head" not in names and names["embed"] == (200, 64) and names["final.norm"] == (64,)
    assert names["l0.mix.in"] == (2 * 96 + 2 * 2 * 16 + 4, 64) and names["l0.mix.conv"] == (96 + 64, 4) and names["l0.mix.conv.b"] == (160,)
    assert names["l0.mix.dt_bias"] == names["l0.mix.A_log"] == names["l0.mix.D"] == (4,) and names["l0.mix.norm"] == (96,)
    assert names["l1.mix.q"] == (32, 64) and names["l1.mix.v"] == (96, 64) and names["l1.mix.a2"] == (4 * 16, 8) and names["l1.mix.dt_bias"] == (64,)
    assert names["l1.mix.g2"] == (96, 16) and names["l1.mix.A_log"] == (4,) and names["l1.mix.norm"] == (24,) and names["l1.mix.b"] == (4, 64)
    assert names["l2.mix.q.b"] == (128,) and names["l2.mix.k.norm"] == (64,) and names["l2.mix.v.b"] == (48,) and names["l2.mix.o.b"] == (64,)
    assert names["l3.mix.g"] == (8, 64) and names["l3.mix.o"] == (64, 8 * 24)
    assert not any(n.startswith(("l3.mix.k", "l3.mix.v")) for n in names) and "l2.norm2" not in names
    assert names["l3.mlp.router.b"] == (5,) and names["l3.mlp.e4.gate"] == (32, 64) and names["l4.mlp.down"] == (64, 56)
    # ranks that a file does not give are the checkpoint's
    raw = copy.deepcopy(CONFIGS["mixed"])
    for key in ("decay_rank", "gate_rank"):
        del raw["layers"][1]["mixer"][key]
    names = {ps.name: tuple(ps.shape) for ps in model_of(raw).param_specs()}
    assert names["l1.mix.a1"] == (None, 64) and names["l1.mix.g2"] == (96, None)


def test_cache_groups_and_state_follow_from_the_mixers():
    model = model_of(CONFIGS["mixed"])
    assert [(g.name, g.layers) for g in model.group_specs] == [("all-2x32v24", 1)]          # layer 3 reads layer 2's pages
    states = {s.name: tuple(s.shape) for s in model.state_specs}
    assert states == {"run0.state": (4, 16, 24), "run0.conv": (3, 160), "run1.state": (4, 16, 24), "run1.conv": (2, 2 * 32 + 96),
                      "run4.state": (6, 24, 16), "run4.conv": (2, 96 + 48)}
    assert all(s.dtype == torch.float32 for s in model.state_specs) and model.graph_safe
    assert {s.name for s in model_of(CONFIGS["bare"]).state_specs} == {"run1.state", "run2.state"}      # one tap: no inputs are kept
    assert model_of(CONFIGS["recurrent"]).group_specs == []


@pytest.mark.parametrize("rot", [
    {"dims": 20, "base": 10000.0, "scaling": {"factor": 6.0, "original": 512, "fast": 32.0, "slow": 1.0}},
    {"dims": 64, "base": 500000.0, "scaling": {"factor": 16.0, "original": 8192, "fast": 20.0, "slow": 2.0}},
    {"dims": 12, "base": 500.0, "scaling": {"factor": 3.0, "original": 64, "fast": 8.0, "slow": 1.0}},
    {"dims": 6, "base": 50.0, "scaling": {"factor": 5.0, "original": 20, "fast": 3.0, "slow": 2.9}},       # the band between is narrow
    {"dims": 8, "base": 100.0, "scaling": {"factor": 2.0, "original": 3, "fast": 32.0, "slow": 0.5}},      # the fast end lies below pair 0
    {"dims": 4, "base": 1.5, "scaling": {"factor": 2.0, "original": 4000, "fast": 1.0, "slow": 0.001}},    # the slow end lies above the last pair
    {"dims": 32, "base": 10000.0},
])
def test_frequencies_stretched_band_by_band(rot):
    from wllm_b200.parts import POSITIONS, spec
    p = POSITIONS.build(spec("rope", theta=rot["base"], head_dim=64, rotary_dim=rot["dims"], exact_table=True, scaling=rot.get("scaling")))
    f, m = plain.frequencies(rot)
    assert p.turn_scale == pytest.approx(m, abs=1e-12) and (m == 1.0) == ("scaling" not in rot)
    assert torch.allclose(p.inv_freq.double(), torch.tensor(f, dtype=torch.float64), rtol=1e-7, atol=0)
    if "scaling" in rot:
        s, full = rot["scaling"], plain.frequencies({"dims": rot["dims"], "base": rot["base"]})[0]
        assert all(1 / s["factor"] - 1e-9 <= a / b <= 1 + 1e-9 for a, b in zip(f, full))      # between divided and kept, in pair order
        assert all(x >= y - 1e-12 for x, y in zip([a / b for a, b in zip(f, full)], [a / b for a, b in zip(f, full)][1:]))


def test_parts_that_do_not_know_the_factor_refuse_it():
    from wllm_b200.parts import MIXERS, spec
    position = spec("rope", theta=1e4, head_dim=16, rotary_dim=16, scaling={"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0})
    base = dict(num_heads=2, num_kv_heads=2, head_dim=16, position=position, q_proj="q", k_proj="k", v_proj="v", o_proj="o")
    kw = dict(hidden_size=32, model_dtype=torch.float32)
    MIXERS.build(spec("attention", **base), **kw)
    with pytest.raises(ValueError, match="turn"):
        MIXERS.build(spec("attention", qk_unit_norm_eps=1e-6, **base), **kw)
    with pytest.raises(ValueError, match="not both"):
        MIXERS.build(spec("attention", sink="s", sink_score=0.0, **base), **kw)
    with pytest.raises(ValueError, match="not both"):
        MIXERS.build(spec("attention", gate_proj="g", head_gate="h", **base), **kw)


def test_the_plain_statements_pieces():
    # a one in the denominator: a row whose scores are all far below zero gives next to nothing, far above zero the usual softmax
    s = torch.tensor([[-50.0, -50.0], [50.0, 50.0], [0.0, 0.0]], dtype=torch.float64)
    p = plain.sink_softmax(s, torch.ones(3, 2, dtype=torch.bool))
    assert p[0].sum() < 1e-20 and p[1].sum() == pytest.approx(1.0) and torch.allclose(p[2], torch.full((2,), 1 / 3, dtype=torch.float64))
    seen = plain.sink_softmax(s, torch.tensor([[True, False]] * 3))
    assert (seen[:, 1] == 0).all()
    # the turn keeps position 0 up to the factor and leaves the rest of a head alone
    rot = {"dims": 4, "base": 100.0, "scaling": {"factor": math.e, "original": 64, "fast": 8.0, "slow": 1.0}}
    x = torch.randn(3, 2, 6, dtype=torch.float64)
    y = plain.turn(x, rot)
    assert torch.allclose(y[0, :, :4], x[0, :, :4] * 1.1) and torch.equal(y[..., 4:], x[..., 4:])
    assert torch.allclose(y[..., :4].norm(dim=-1), x[..., :4].norm(dim=-1) * 1.1)
    # a short convolution: the last tap is the token's own
    x = torch.arange(1.0, 6.0)[:, None]
    assert plain.short_conv(x, torch.tensor([[100.0, 10.0, 1.0]]), torch.tensor([0.5]))[:, 0].tolist() == [1.5, 12.5, 123.5, 234.5, 345.5]
    # a state space that does not forget adds dt B x up and reads it with C
    one = torch.ones(3, 1, 1, dtype=torch.float64)
    y = plain.ssd(one, one * 2, one * 3, torch.full((3, 1), 0.5, dtype=torch.float64), torch.zeros(1, dtype=torch.float64), torch.tensor([10.0], dtype=torch.float64))
    assert y[:, 0, 0].tolist() == [13.0, 16.0, 19.0]
    # the delta rule without decay and with a full step stores v along k, and overwrites it
    e = torch.eye(2, dtype=torch.float64)
    k = torch.stack([e[0], e[1], e[0]])[:, None]
    v = torch.tensor([[5.0], [7.0], [9.0]], dtype=torch.float64)[:, None]
    o = plain.delta_steps(k, k, v, torch.ones(3, 1, dtype=torch.float64), torch.ones(3, 1, 2, dtype=torch.float64))
    assert o[:, 0, 0].tolist() == [5.0, 7.0, 9.0]
    g = torch.ones(3, 1, 2, dtype=torch.float64)
    g[1, 0, 0] = 0.5                                    # the channel of e_0 forgets half before the second token
    o = plain.delta_steps(torch.stack([e[0], e[0], e[0]])[:, None], k, v, torch.ones(3, 1, dtype=torch.float64), g)
    assert o[:, 0, 0].tolist() == [5.0, 2.5, 9.0]
    # the experts' weights are the softmax over the chosen logits, which carry the bias
    w = {"router": torch.zeros(3, 2, dtype=torch.float64), "router.b": torch.tensor([0.0, 1.0, 3.0], dtype=torch.float64)}
    idx, weight = plain.route({"router": {"top": 2}}, w, "", torch.zeros(1, 2, dtype=torch.float64))
    assert idx.tolist() == [[2, 1]] and weight[0, 0] == pytest.approx(1 / (1 + math.exp(-2)))
