"""Tebozen without a GPU: configuration, plan, what the cache is asked for, and the plain implementation's own mechanisms
against closed forms."""
import copy
import math

import numpy as np
import pytest

import plain_tebozen as pz
import tebozen_helpers as th
import questwend_b200  # noqa: F401
from questwend_b200.config import ConfigError
from questwend_b200.config.registry import config_from_dict, get_architecture
from questwend_b200.parts.base import KVSpec, StateSpec


def plan_of(cfgd):
    return get_architecture("Tebozen").plan(config_from_dict(cfgd))


def test_config_reads_every_size_and_round_trips():
    cfg = config_from_dict(th.MIXED)
    assert cfg.architecture == "Tebozen" and (cfg.width, cfg.vocab, cfg.norm_eps, cfg.embedding_scale) == (64, 90, 2e-5, 1.7)
    assert cfg.layers[1]["mixer"] == {"dim": 8, "gate_cap": 4.0, "heads": 3, "vdim": 12}
    assert cfg.layers[2]["mixer"] == {"conv": 3, "diff": 0.3, "dim": 16, "heads": 4, "kv_heads": 2, "mask": {"size": 20}, "scale": 0.4,
                                      "rot": {"base": 300.0, "dims": 8}, "vdim": 24}
    assert [l["mixer"].get("kv_from") for l in cfg.layers] == [None, None, None, 0, None, None, None, None, 6, 0]
    assert cfg.layers[3]["mlp"] is None and cfg.layers[6]["mlp"]["shared"] is None and cfg.layers[1]["mlp"]["router"] == {"experts": 9, "top": 4}
    for d in (th.MIXED, th.ONES):
        c = config_from_dict(d)
        assert c.to_dict() == d and config_from_dict(c.to_dict()) == c
    bare = copy.deepcopy(th.MIXED)
    del bare["layers"][2]["mixer"]["mask"], bare["embedding"]
    c = config_from_dict(bare)
    assert c.layers[2]["mixer"]["mask"] is None and c.embedding_scale == 1.0 and config_from_dict(c.to_dict()) == c


@pytest.mark.parametrize("path, value, word", [
    (("layers", 0, "type"), "conv", "'type'"), (("layers", 2, "mixer", "kv_heads"), 3, "'heads'"), (("layers", 2, "mixer", "dim"), 300, "'dim'"),
    (("layers", 2, "mixer", "conv"), 17, "'conv'"), (("layers", 2, "mixer", "conv"), 0, "'conv'"), (("layers", 2, "mixer", "mask", "size"), 0, "'size'"),
    (("layers", 2, "mixer", "rot", "dims"), 18, "'dims'"), (("layers", 2, "mixer", "rot", "dims"), 3, "'dims'"), (("layers", 2, "mixer", "rot", "base"), 1.0, "'base'"),
    (("layers", 1, "mixer", "dim"), 513, "'dim'"), (("layers", 1, "mixer", "gate_cap"), 0, "'gate_cap'"), (("layers", 0, "mixer", "kv_rank"), 513, "'kv_rank'"),
    (("layers", 0, "mixer", "scale"), 0.0, "'scale'"), (("layers", 0, "mlp", "kind"), "dense", "'kind'"), (("layers", 0, "mlp", "router", "top"), 7, "'top'"),
    (("layers", 3, "mixer", "kv_from"), 3, "'kv_from'"), (("layers", 3, "mixer", "kv_from"), 1, "'kv_from'"), (("layers", 9, "mixer", "kv_from"), 3, "'kv_from'"),
    (("layers", 8, "mixer", "kv_from"), 0, "'kv_rank'"), (("layers", 8, "mixer", "rot", "base"), 91.0, "'rot'"), (("layers", 3, "mixer", "kv_rank"), 32, "'kv_rank'"),
    (("norm", "eps"), 0.0, "'eps'"), (("vocab",), 0, "'vocab'")])
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
    # a layer without a feed-forward may have its second norm in the files: it is not used
    assert [t.ignored for t in plan_of(th.MIXED).manifest() if t.name == "l3.norm2"] == [True]


def test_what_the_cache_is_asked_for():
    import torch
    from questwend_b200.cache import CacheManager
    from questwend_b200.engine.model import Model
    from questwend_b200.parts.base import Runtime
    model = Model(plan_of(th.MIXED), Runtime(torch.device("cpu"), torch.float32))
    units = model.cache_units()
    assert units[0] == (KVSpec(1, 48, 0, values=False), None, None) and units[3][2] == 0 and units[8][2] == 6 and units[9][2] == 0
    assert units[1] == (None, (StateSpec((3, 13, 8)), StateSpec((3, 13))), None)
    assert units[2] == (KVSpec(2, 32, 20, value_dim=24), StateSpec((2, 4 * 32 + 2 * 32 + 2 * 24)), None)
    assert units[7] == (KVSpec(2, 64, 130, value_dim=8), None, None)            # one tap has no tail
    assert "mlstm" in model.kernel_modules() and "moe" in model.kernel_modules()
    cache = CacheManager(units, 200, 2, 200, torch.float32, "cpu")
    own, shared, other = cache.unit_cache(0), cache.unit_cache(9), cache.unit_cache(6)
    assert shared.k_pool.data_ptr() == own.k_pool.data_ptr() != other.k_pool.data_ptr()
    assert own.writable and not shared.writable and shared.group_id == own.group_id
    state, m = cache.unit_cache(1).state
    (s,) = cache.open(1)
    state.fill_(3.0), m.fill_(2.0)
    cache.close([s])
    assert cache.open(1) == [s] and not state[s].any() and not m[s].any() and state[1 - s].all()    # a slot starts from zeros


def test_random_weights_folder_round_trips(tmp_path):
    import questwend_b200 as qw
    from questwend_b200.config.registry import load_config
    from questwend_b200.weights.safetensors_io import SafetensorsFolder
    cfg = config_from_dict(th.MIXED)
    qw.write_model_folder(str(tmp_path), cfg, seed=3, dtype="bfloat16")
    assert load_config(str(tmp_path)) == cfg
    folder = SafetensorsFolder(str(tmp_path))
    assert folder.tensor("l0.norm1").float().abs().max() <= 0.1 and folder.tensor("l1.mix.norm").float().min() >= 0.89
    folder.close()


def test_parts_refuse_what_they_cannot_do():
    import torch
    from questwend_b200.parts import PartSpec, Runtime, build_part
    rt = Runtime(torch.device("cpu"), torch.float32)
    memory = {"hidden_size": 16, "heads": 1, "key_dim": 8, "vdim": 8, "gate_cap": 5.0, "norm_eps": 1e-5}
    build_part("mixer", PartSpec("mlstm", memory), rt, position=None)
    for change in ({"gate_cap": 0.0}, {"key_dim": 600}, {"vdim": 0}):
        with pytest.raises(ValueError):
            build_part("mixer", PartSpec("mlstm", {**memory, **change}), rt, position=None)
    with pytest.raises(ValueError):
        build_part("feed_forward", PartSpec("routed_experts", {"hidden_size": 16, "expert_size": 8, "experts": 2, "top": 1, "gated": False,
                                                               "activation": "relu2", "weight_on": "both"}), rt)


# ----------------------------------------------------------------------------- the plain implementation's mechanisms
def test_plain_matrix_memory():
    q, k, v = np.array([[1.0], [2.0], [1.0]]), np.array([[1.0], [-1.0], [0.5]]), np.array([[3.0, 1.0], [5.0, 0.0], [0.0, 2.0]])
    i, f = np.array([-1.0, 2.0, 0.0]), np.array([-0.5, -1.0, -0.25])
    out = pz.matrix_memory(q, k, v, i, f)
    # the memory itself, without a running maximum: S e^m and n e^m, and a floor of 1 on |n q| e^m; only `TINY` knows of m
    S, n, m = np.zeros(2), 0.0, 0.0
    for t in range(3):
        S, n = math.exp(f[t]) * S + math.exp(i[t]) * k[t, 0] * v[t], math.exp(f[t]) * n + math.exp(i[t]) * k[t, 0]
        m = max(f[t] + m, i[t])
        assert np.allclose(out[t], S * q[t, 0] / (max(abs(n * q[t, 0]), 1.0) + pz.TINY * math.exp(m)), rtol=1e-12)
    # the maximum starts at 0: a small first write stays small (from minus infinity it would be normalised away)
    assert np.allclose(pz.matrix_memory(np.ones((1, 1)), np.ones((1, 1)), np.ones((1, 1)), np.array([-4.0]), np.array([-1.0])), math.exp(-4.0), rtol=1e-4)


def test_plain_gates_turn_window_and_convolution():
    m = {"gate_cap": 3.0}
    w = {"i": np.array([[2.0]]), "i.b": np.array([1.0]), "f": np.array([[1.0]]), "f.b": np.array([0.5])}
    i, f = pz.gates(np.array([[1.5], [100.0]]), m, w, "")
    assert np.allclose(i[:, 0], [3 * math.tanh(4 / 3), 3.0])
    assert np.allclose(f[:, 0], [-math.log1p(math.exp(-3 * math.tanh(2 / 3))), -math.log1p(math.exp(-3.0))])
    x = np.arange(1.0, 7.0)[None, :].repeat(2, 0)
    for neighbours, pairs in ((False, ((0, 2), (1, 3))), (True, ((0, 1), (2, 3)))):
        out = pz.turn(x, [0, 5], 100.0, 4, neighbours)
        assert np.allclose(out[0], x[0]) and np.allclose(out[1, 4:], x[1, 4:])
        for p, (a, b) in enumerate(pairs):
            g = 5 * 100.0 ** (-2 * p / 4)
            assert np.allclose([out[1, a], out[1, b]], [x[1, a] * math.cos(g) - x[1, b] * math.sin(g), x[1, b] * math.cos(g) + x[1, a] * math.sin(g)])
    seen = pz.visible(6, 2)
    assert seen.sum() == 11 and seen[4, 4] and seen[4, 3] and not seen[4, 2] and not seen[3, 4]
    assert np.allclose(pz.conv_over_time(np.array([[1.0], [2.0], [4.0]]), np.array([[10.0, 1.0]]))[:, 0], [1.0, 12.0, 24.0])


def test_plain_experts_see_weighted_inputs():
    rng = np.random.default_rng(0)
    h, w = rng.standard_normal((5, 6)), {"e.up": rng.standard_normal((4, 6)), "e.down": rng.standard_normal((6, 4))}
    s = np.array([[0.3], [0.9], [0.5], [1.0], [0.1]])
    assert np.allclose(pz.expert(h, w, "e.", weight=s), pz.expert(h * s, w, "e."))
    assert np.allclose(pz.expert(h, w, "e.", weight=s), s ** 2 * pz.expert(h, w, "e."))         # relu squared: not s times
    chosen, weights = pz.route(np.array([[0.0, 2.0, -1.0, 2.0]]), 3)
    assert chosen.tolist() == [[1, 3, 0]] and np.allclose(weights, [[pz.sigmoid(2.0), pz.sigmoid(2.0), 0.5]])


def test_plain_difference_weight():
    w = {"lq1": np.array([1.0, 0.5]), "lk1": np.array([0.5, 1.0]), "lq2": np.array([0.0, 2.0]), "lk2": np.array([3.0, -0.5])}
    assert np.isclose(pz.difference_weight(w, "", 0.25), math.exp(1.0) - math.exp(-1.0) + 0.25)
