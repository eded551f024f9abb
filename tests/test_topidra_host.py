"""Host side of Topidra and its oracle, without a GPU: configuration, tensor shapes, layer runs, and properties that pin the oracle."""
import json

import numpy as np
import pytest

from nn_b200 import registry
from nn_b200.topidra import TopidraConfig
from nn_b200.weights import InvalidDataError, SafeTensors, check_shapes, write_safetensors
from oracle import topidra as F
from tests.fabezen_models import wide64
from tests.topidra_models import CONFIGS, attention, config, lightning, weights_for


def test_configuration_and_shapes():
    cfg = TopidraConfig.from_dict(CONFIGS["mixed"])
    shapes = cfg.tensor_shapes()
    assert shapes["head"] == (103, 60) and shapes["l1.mix.q"] == (120, 60) and shapes["l1.mix.k"] == (40, 60) and shapes["l1.mix.v"] == (56, 60)
    assert shapes["l1.mix.q.norm"] == (120,) and shapes["l1.mix.g"] == (6, 60) and shapes["l0.mix.g"] == (108, 60) and shapes["l0.mix.norm"] == (108,)
    assert "l0.norm2b" in shapes and "l2.norm2" not in shapes and "l3.mlp.up" not in shapes
    for bad in (config([]), config([{**lightning(), "type": "other"}]), config([lightning()], loop=(0, 2, 1)), config([lightning()], loop=(1, 0, 2)),
                config([lightning()], loop=(0, 1, 0))):
        with pytest.raises(ValueError):
            TopidraConfig.from_dict(bad)


def test_runs_of_a_loop():
    layers = [lightning()] * 4
    assert TopidraConfig.from_dict(config(layers)).runs() == [(i, False) for i in range(4)]
    for loop, order, again in (((1, 3, 3), [0, 1, 2, 1, 2, 1, 2, 3], [3, 5]), ((0, 4, 2), [0, 1, 2, 3] * 2, [4]), ((2, 2, 5), [0, 1, 2, 3], []),
                               ((3, 4, 2), [0, 1, 2, 3, 3], [4])):
        runs = TopidraConfig.from_dict(config(layers, loop=loop)).runs()
        assert [i for i, _ in runs] == order and [n for n, (_, a) in enumerate(runs) if a] == again
        assert runs == F.runs(config(layers, loop=loop))


def test_model_folder(tmp_path):
    cfg = CONFIGS["ones"]
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    w = weights_for(cfg, 1)
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    assert registry.read_config(str(tmp_path))["architecture"] in registry.ARCHITECTURES
    model_class, config_class = registry.ARCHITECTURES["Topidra"]()
    got = SafeTensors(str(tmp_path / "model.safetensors"))
    check_shapes(got, config_class.from_dict(cfg).tensor_shapes())
    del w["l0.mix.sink"]
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    with pytest.raises(InvalidDataError, match="l0.mix.sink"):
        check_shapes(SafeTensors(str(tmp_path / "model.safetensors")), config_class.from_dict(cfg).tensor_shapes())


# ---------------------------------------------------------------------------------------------- the oracle
def test_sink_takes_its_share():
    a = F.sink_softmax(np.zeros((2, 3, 3)), np.array([0.0, -1e9]), F.visible(range(3), range(3), 2))
    assert np.allclose(a[0], [[1 / 2, 0, 0], [1 / 3, 1 / 3, 0], [0, 1 / 3, 1 / 3]]) and np.allclose(a[1], [[1, 0, 0], [.5, .5, 0], [0, .5, .5]])
    big = F.sink_softmax(np.zeros((1, 1, 1)), np.array([800.0]), np.ones((1, 1), bool))
    assert big[0, 0, 0] == 0.0


def test_window_counts_its_own_position():
    assert F.visible([5], range(8), 3).tolist() == [[False, False, False, True, True, True, False, False]]
    assert F.visible([0], [0], 1).tolist() == [[True]]


def test_decayed_memory_by_hand_and_in_pieces():
    q = k = np.ones((3, 1, 1))
    v = np.array([1.0, 10.0, 100.0]).reshape(3, 1, 1)
    assert F.decayed_memory(q, k, v, [0.5])[0].ravel().tolist() == [1.0, 10.5, 105.25]
    assert F.decayed_memory(q, k, v, [0.0])[0].ravel().tolist() == [1.0, 10.0, 100.0]
    rng = np.random.default_rng(0)
    q, k, v, d = rng.standard_normal((9, 2, 4)), rng.standard_normal((9, 2, 4)), rng.standard_normal((9, 2, 3)), [0.7, 1.0]
    o, s = F.decayed_memory(q, k, v, d)
    o1, s1 = F.decayed_memory(q[:5], k[:5], v[:5], d)
    o2, s2 = F.decayed_memory(q[5:], k[5:], v[5:], d, s1)
    assert np.allclose(np.concatenate([o1, o2]), o) and np.allclose(s2, s)


@pytest.mark.parametrize("name", list(CONFIGS))
def test_the_oracle_is_causal(name):
    cfg = CONFIGS[name]
    w = wide64(weights_for(cfg, 1))
    t = np.random.default_rng(4).integers(0, cfg["vocab"], 12)
    full = F.forward(t, w, cfg)
    t2 = t.copy()
    t2[8:] = (t2[8:] + 1) % cfg["vocab"]
    assert np.allclose(F.forward(t2, w, cfg)[:8], full[:8]) and not np.allclose(F.forward(t2, w, cfg)[8], full[8])


def test_a_loop_is_its_layers_written_out():
    cfg = config([lightning(), attention(), lightning(ff=8)], loop=(1, 2, 3))
    w = wide64(weights_for(cfg, 2))
    t = np.arange(7)
    x = w["embed"][t]
    x = F.layer(x, w, "l0.", cfg["layers"][0], 3e-5)
    for p in range(3):
        x = F.layer(x + (w["embed"][t] if p else 0.0), w, "l1.", cfg["layers"][1], 3e-5)
    x = F.layer(x, w, "l2.", cfg["layers"][2], 3e-5)
    assert np.allclose(F.forward(t, w, cfg), F.rms_norm(x, w["final.norm"], 3e-5) @ w["head"].T)
