"""Host side of Fabezen and its oracle, without a GPU: configuration, tensor shapes, model folders, registry, and properties that
pin the oracle itself."""
import json

import numpy as np
import pytest

from nn_b200.blocks import bf16_bits, f32
from nn_b200.fabezen import FabezenConfig
from nn_b200.registry import load_model
from nn_b200.weights import InvalidDataError, SafeTensors, check_shapes, write_safetensors
from oracle import fabezen as F
from tests.fabezen_models import CONFIGS, config, delta, latent, weights_for, wide64


def test_safetensors_round_trip_and_errors(tmp_path):
    path = str(tmp_path / "m.safetensors")
    t = {"a": np.arange(6, dtype=np.float32).reshape(2, 3), "b": np.array([1, 2, 3], np.uint16), "c": np.array([-1, 5], np.int32), "empty": np.empty((0, 4), np.float32)}
    write_safetensors(path, t)
    got = SafeTensors(path)
    assert sorted(got) == sorted(t)
    for k in t:
        assert got[k].shape == t[k].shape and np.array_equal(got[k], t[k])
    check_shapes(got, {"a": (2, None), "b": (3,)})
    with pytest.raises(InvalidDataError, match="missing"):
        check_shapes(got, {"z": (1,)})
    with pytest.raises(InvalidDataError, match="Shape mismatch"):
        check_shapes(got, {"a": (3, 2)})
    data = open(path, "rb").read()
    for bad in (b"", data[:6], data[:-4], b"\xff" * 16):
        open(path, "wb").write(bad)
        with pytest.raises(InvalidDataError):
            SafeTensors(path)


def test_an_odd_header_length_is_read(tmp_path):
    """Tensor data need not start on a multiple of its element size."""
    head = json.dumps({"x": {"dtype": "F32", "shape": [2], "data_offsets": [1, 9]}}).encode()
    path = str(tmp_path / "m.safetensors")
    with open(path, "wb") as f:
        f.write(len(head).to_bytes(8, "little") + head + b"\0" + np.array([1.5, -2.0], "<f4").tobytes())
    assert list(SafeTensors(path)["x"]) == [1.5, -2.0]


def test_configuration():
    cfg = FabezenConfig.from_dict(CONFIGS["mixed"])
    assert [cfg.owner(i) for i in range(6)] == [0, 1, 2, 0, 4, 2]
    shapes = cfg.tensor_shapes()
    assert "l3.norm1" not in shapes and "l4.norm2" not in shapes and shapes["bigram"] == (38, 60)
    chain = FabezenConfig.from_dict(config([delta(), delta(weights_of=0), delta(weights_of=1)]))
    assert chain.owner(2) == 0
    with pytest.raises(ValueError):
        FabezenConfig.from_dict(config([delta(weights_of=3)]))
    with pytest.raises(ValueError):
        FabezenConfig.from_dict(config([{**delta(), "type": "other"}]))
    with pytest.raises(ValueError):
        FabezenConfig.from_dict(config([delta(weights_of=1), delta(weights_of=0)])).owner(0)


def test_registry_refuses_what_it_does_not_know(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Unknown"}))
    with pytest.raises(ValueError, match="Unknown"):
        load_model(None, str(tmp_path))
    with pytest.raises(ValueError, match="float16"):
        load_model(None, str(tmp_path), "float16")


def test_bf16_bits_round_to_nearest_even():
    x = np.array([1.0, 1.00390625, 1.01171875, -3.14159], np.float32)        # the second and third lie halfway
    assert np.array_equal(f32(bf16_bits(x)), np.array([1.0, 1.0, 1.015625, -3.140625], np.float32))


# ---------------------------------------------------------------------------------------------- the oracle
def test_delta_rule_stores_and_overwrites():
    """Without decay and with beta 1 the state answers a key with the last value written under it."""
    k = np.eye(4)[[0, 1, 0]][:, None, :]
    v = np.random.default_rng(0).standard_normal((3, 1, 5))
    o, s = F.delta_rule(k, k, v, np.ones((3, 1)), np.ones((3, 1, 4)))
    assert np.allclose(o, v) and np.allclose(s[0, 0], v[2, 0]) and np.allclose(s[0, 1], v[1, 0])
    o2, _ = F.delta_rule(k[2:], k[2:], v[2:], np.ones((1, 1)), np.ones((1, 1, 4)), F.delta_rule(k[:2], k[:2], v[:2], np.ones((2, 1)), np.ones((2, 1, 4)))[1])
    assert np.allclose(o2, o[2:])


def test_rotation_keeps_relative_positions():
    rng = np.random.default_rng(1)
    a, b = rng.standard_normal((1, 8)), rng.standard_normal((1, 8))
    dot = lambda p, q: float((F.rotate(a, [p], 100.0, 6) * F.rotate(b, [q], 100.0, 6)).sum())
    assert dot(5, 2) == pytest.approx(dot(13, 10)) and dot(5, 2) != pytest.approx(dot(5, 3))


def test_window_of_one_returns_the_own_value():
    v = np.random.default_rng(2).standard_normal((4, 2, 3))
    assert np.allclose(F.windowed_softmax_attention(np.random.default_rng(3).standard_normal((2, 4, 4)), v, 1), v)


def test_short_convolution_by_hand():
    x, taps = np.array([[1.0], [2.0], [3.0]]), np.array([[10.0, 100.0]])
    assert np.allclose(F.short_conv(x, taps)[:, 0], F.silu(np.array([100.0, 210.0, 320.0])))


@pytest.mark.parametrize("name", list(CONFIGS))
def test_the_oracle_is_causal(name):
    cfg = CONFIGS[name]
    w = wide64(weights_for(cfg, 1))
    t = np.random.default_rng(4).integers(0, cfg["vocab"], 12)
    full = F.forward(t, w, cfg)
    t2 = t.copy()
    t2[8:] = (t2[8:] + 1) % cfg["vocab"]
    assert np.allclose(F.forward(t2, w, cfg)[:8], full[:8]) and not np.allclose(F.forward(t2, w, cfg)[8], full[8])


def test_bigram_rows():
    assert F.bigram_rows([3, 4, 9], 7, 2, 5) == [7, (3 * 2 + 4 * 5) % 7, (4 * 2 + 9 * 5) % 7]
