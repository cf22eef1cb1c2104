"""Tufadra without a GPU: configuration, plan, what the cache is asked for, and the plain implementation's own
mechanisms against closed forms."""
import copy
import math

import numpy as np
import pytest

import plain_tufadra as pt
import tufadra_helpers as th
import questwend_b200  # noqa: F401
from questwend_b200.config import ConfigError
from questwend_b200.config.registry import config_from_dict, get_architecture
from questwend_b200.parts.base import KVSpec


def plan_of(cfgd):
    return get_architecture("Tufadra").plan(config_from_dict(cfgd))


def test_config_reads_every_size_and_round_trips():
    cfg = config_from_dict(th.MIXED)
    assert cfg.architecture == "Tufadra" and cfg.width == 64 and cfg.vocab == 96 and cfg.norm_eps == 2e-5 and cfg.max_positions == 700
    assert cfg.layers[0]["mixer"] == {"dim": 24, "heads": 6, "kv_heads": 2, "scale": 0.3, "vdim": 40, "q_temp": {"coef": 0.7, "every": 10}}
    assert cfg.layers[2]["mlp"]["router"] == {"experts": 12, "groups": {"count": 2, "keep": 1}, "scale": 2.0, "top": 5}
    assert cfg.layers[1]["mlp"] is None and cfg.layers[4]["mlp"]["shared"] == {"ff": 30}
    assert [cfg.tensors_of(i) for i in range(8)] == [0, 1, 2, 0, 4, 1, 6, 0]
    for d in (th.MIXED, th.ONES):
        c = config_from_dict(d)
        assert c.to_dict() == d and config_from_dict(c.to_dict()) == c
    bare = copy.deepcopy(th.MIXED)
    for entry in bare["layers"]:
        if entry["mlp"]:
            entry["mlp"].pop("shared", None)
            entry["mlp"]["router"].pop("groups", None)
    c = config_from_dict(bare)
    assert c.layers[0]["mlp"]["shared"] is None and c.layers[0]["mlp"]["router"]["groups"] == {"count": 1, "keep": 1}
    assert config_from_dict(c.to_dict()) == c
    names = {t.name for t in plan_of(bare).manifest()}
    assert "l0.mlp.router" in names and "l0.mlp.shared.up" not in names and "l0.mlp.shared.sg" not in names


@pytest.mark.parametrize("path, value, word", [
    (("layers", 0, "type"), "conv", "'type'"), (("layers", 2, "mixer", "kv_heads"), 2, "'heads'"),
    (("layers", 0, "mixer", "dim"), 264, "'dim'"), (("layers", 1, "mixer", "vdim"), 0, "'vdim'"),
    (("layers", 0, "mixer", "q_temp", "every"), 0, "'every'"), (("layers", 0, "mixer", "scale"), 0.0, "'scale'"),
    (("layers", 0, "mlp", "kind"), "dense", "'kind'"), (("layers", 2, "mlp", "router", "top"), 7, "groups"),
    (("layers", 2, "mlp", "router", "groups", "count"), 5, "groups"), (("layers", 2, "mlp", "router", "groups", "keep"), 3, "groups"),
    (("layers", 2, "mlp", "router", "top"), 17, "'top'"), (("layers", 2, "mlp", "router", "experts"), 2048, "experts"),
    (("layers", 3, "weights_of"), 8, "'weights_of'"), (("layers", 3, "weights_of"), 3, "'weights_of'"),
    (("layers", 0, "weights_of"), 7, "'weights_of'"), (("layers", 3, "weights_of"), 1, "'weights_of'"),
    (("max_positions",), 0, "'max_positions'"), (("norm", "eps"), 0.0, "'eps'")])
def test_config_refuses_with_the_keys_name(path, value, word):
    bad = copy.deepcopy(th.MIXED)
    at = bad
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    with pytest.raises(ConfigError) as e:
        config_from_dict(bad)
    assert word in str(e.value)


def test_manifest_names_and_shapes():
    for cfgd in (th.MIXED, th.ONES):
        w = th.draw_weights(cfgd)
        shapes = {t.name: tuple(t.shape) for t in plan_of(cfgd).manifest() if not t.ignored}
        assert shapes == {k: v.shape for k, v in w.items()}


def test_a_layer_that_is_run_twice_has_one_set_of_tensors_and_two_caches():
    import torch
    from questwend_b200.engine.model import Model
    from questwend_b200.parts.base import Runtime
    plan = plan_of(th.MIXED)
    assert [run.layer for run in plan.schedule] == [0, 1, 2, 0, 3, 1, 4, 0] and len(plan.layers) == 5
    assert plan.position_limit == plan.max_position == 700
    model = Model(plan, Runtime(torch.device("cpu"), torch.bfloat16))
    units = model.cache_units()
    assert [u[0] for u in units] == [KVSpec(2, 24, 0, value_dim=40), KVSpec(4, 16, 0, value_dim=16), KVSpec(1, 40, 0, value_dim=8),
                                     KVSpec(2, 24, 0, value_dim=40), KVSpec(1, 64, 0, value_dim=64), KVSpec(4, 16, 0, value_dim=16),
                                     KVSpec(1, 12, 0, value_dim=20), KVSpec(2, 24, 0, value_dim=40)]
    assert all(u[1] is None and u[2] is None for u in units)
    assert "attention_tc" in model.kernel_modules() and "moe" in model.kernel_modules()
    cfgd = th.config([(th.attention(), None), (th.attention(), None)])
    cfgd["layers"][0]["weights_of"] = 1                     # an entry may name a later layer as well
    plan = plan_of(cfgd)
    assert [run.layer for run in plan.schedule] == [0, 0] and plan.layers[0].block.prefix == "l1."


def test_random_weights_folder_round_trips(tmp_path):
    import questwend_b200 as qw
    from questwend_b200.config.registry import load_config
    from questwend_b200.weights.safetensors_io import SafetensorsFolder
    cfg = config_from_dict(th.MIXED)
    qw.write_model_folder(str(tmp_path), cfg, seed=3, dtype="bfloat16")
    assert load_config(str(tmp_path)) == cfg
    folder = SafetensorsFolder(str(tmp_path))
    assert folder.tensor("l0.norm1").float().abs().max() <= 0.1 and folder.tensor("l0.mix.q.norm").float().min() >= 0.89
    folder.close()


def test_the_router_part_refuses_what_it_cannot_choose():
    import torch
    from questwend_b200.parts import PartSpec, Runtime, build_part
    ok = {"hidden_size": 16, "expert_size": 8, "experts": 8, "top": 2, "gated": False, "activation": "gelu", "scores": "sigmoid"}
    for change in ({"groups": 3}, {"groups": 4, "groups_kept": 5}, {"groups": 4, "groups_kept": 1, "top": 3}, {"scores": "tanh"},
                   {"activation": "xielu"}, {"gated": True, "shared_size": 8}):
        with pytest.raises(ValueError):
            build_part("feed_forward", PartSpec("routed_experts", {**ok, **change}), Runtime(torch.device("cpu"), torch.float32))
    build_part("feed_forward", PartSpec("routed_experts", ok), Runtime(torch.device("cpu"), torch.float32))


# ----------------------------------------------------------------------------- the plain implementation's mechanisms
def test_plain_query_temperature_and_gelu():
    f = pt.query_temperature([0, 8, 9, 18, 19, 99], 0.5, 10)
    assert np.allclose(f, [1.0, 1.0, 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(3), 1 + 0.5 * math.log(11)])
    assert np.allclose(pt.query_temperature([0, 1, 2], 1.0, 1), 1.0 + np.log([2.0, 3.0, 4.0]))
    assert np.allclose(pt.gelu_exact([1.0, -1.0, 0.0]), [0.8413447460685429, -0.15865525393145707, 0.0])


def test_plain_norms():
    x = np.array([[3.0, 4.0]])
    assert np.allclose(pt.norm_about_one(x, np.array([0.0, 1.0]), 0.0), x / math.sqrt(12.5) * np.array([1.0, 2.0]))
    m = {"heads": 2, "kv_heads": 1, "dim": 1, "vdim": 1, "scale": 1.0, "q_temp": {"coef": 0.0, "every": 1}}
    w = {"q": np.array([[1.0, 0.0], [0.0, 2.0]]), "k": np.array([[1.0, 1.0]]), "v": np.array([[1.0, -1.0]]), "q.norm": np.array([2.0, 1.0]),
         "k.norm": np.array([1.0]), "o": np.eye(2)}
    h = np.array([[1.0, 1.0], [1.0, -3.0]])
    got = pt.attention(h, m, w, "", 0.0)
    # token 1: q = (1, -6) / sqrt(37/2) * (2, 1); keys sign(2), sign(-2); values 0 and 4
    q = np.array([1.0, -6.0]) / math.sqrt(37 / 2) * np.array([2.0, 1.0])
    assert np.allclose(got[0], 0.0)
    for hd in range(2):
        e = np.exp([q[hd], -q[hd]])
        assert np.isclose(got[1, hd], 4.0 * e[1] / e.sum())


def test_plain_router():
    router = {"experts": 6, "top": 2, "scale": 2.0, "groups": {"count": 3, "keep": 1}}
    z = np.array([[0.0, 0.0, 3.0, -2.0, 1.0, 1.0]])
    s = pt.sigmoid(z[0])
    chosen, weights = pt.route(z, np.zeros(6), router)
    assert chosen.tolist() == [[4, 5]]                      # 2 x 0.731 beats 0.953 + 0.119
    assert np.allclose(weights, 1.0)
    c = np.array([-3.0, -3.0, -9.0, -9.0, -9.0, -9.0])      # all choice scores negative: the masked experts must still lose
    chosen, weights = pt.route(z, c, router)
    assert chosen.tolist() == [[0, 1]] and np.allclose(weights, 1.0)
    router = {"experts": 6, "top": 3, "scale": 1.0, "groups": {"count": 3, "keep": 2}}
    chosen, weights = pt.route(z, np.array([0.0, 0, 0, 0, 0, 0.5]), router)
    assert chosen.tolist() == [[5, 2, 4]]
    assert np.allclose(weights[0], s[chosen[0]] / s[chosen[0]].sum())
    ones = {"experts": 3, "top": 1, "scale": 1.5, "groups": {"count": 3, "keep": 2}}     # groups of one expert
    assert pt.route(np.array([[0.0, 2.0, 1.0]]), np.zeros(3), ones)[0].tolist() == [[1]]
