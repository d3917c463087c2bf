"""Models described layer by layer, the parts that need no GPU: the plain implementation against itself,
configuration reading, the safetensors reader."""
import json
import os

import numpy as np
import pytest

import layered_models as LM
import plain_layered as P
import strict_b200 as sb
from strict_b200 import checkpoint


def test_rotation_keeps_lengths_and_depends_on_distance_only():
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal((2, 1, 12))
    at = lambda x, p: P.rotate_interleaved(x, np.array([p]), 300.0, 8)[0]  # noqa: E731
    assert np.allclose(np.linalg.norm(at(q, 17)), np.linalg.norm(q)) and np.array_equal(at(q, 5)[8:], q[0, 8:])
    assert np.allclose(at(q, 30) @ at(k, 10), at(q, 120) @ at(k, 100)) and not np.allclose(at(q, 30) @ at(k, 10), at(q, 30) @ at(k, 11))
    one = P.rotate_interleaved(np.array([[1.0, 0.0, 0.0, 1.0]]), np.array([2]), 100.0, 4)[0]
    assert np.allclose(one, [np.cos(2), np.sin(2), -np.sin(0.2), np.cos(0.2)])


def test_group_norm_of_one_group_is_the_rms_norm():
    x = np.random.default_rng(1).standard_normal((3, 12))
    w = np.arange(12.0)
    assert np.allclose(P.group_rms_norm(x, w, 1e-5, 1), P.rms_norm(x, w, 1e-5))
    y = P.group_rms_norm(x, np.ones(12), 0.0, 3).reshape(3, 3, 4)
    assert np.allclose((y * y).mean(-1), 1.0)


def test_window_counts_the_position_itself():
    m = P.visible(3, 8, 5, 3)
    assert m[0].nonzero()[0].tolist() == [3, 4, 5] and m[2].nonzero()[0].tolist() == [5, 6, 7]
    assert P.visible(1, 8, 5, None)[0].nonzero()[0].tolist() == list(range(6))


def test_xielu_is_smooth_at_zero():
    p, q = 0.3, -0.7
    e = 1e-6
    assert P.xielu(np.array(0.0), p, q) == 0 and abs(float((P.xielu(np.array(e), p, q) - P.xielu(np.array(-e), p, q)) / (2 * e)) - 0.5) < 1e-5
    assert np.isclose(P.xielu(np.array(2.0), p, q), np.log1p(np.exp(p)) * 4 + 1)
    assert np.isclose(P.xielu(np.array(-2.0), p, q), (0.5 + np.log1p(np.exp(q))) * (np.exp(-2) - 1 + 2) - 1)


def test_plain_model_is_causal_and_the_window_binds():
    cfg = LM.CONFIGS["ragged"]
    w = LM.weights(cfg, 3)
    t = np.random.default_rng(4).integers(0, cfg["vocab"], 40)
    full = P.forward(cfg, w, t)
    assert np.allclose(full[:25], P.forward(cfg, w, t[:25]))
    other = json.loads(json.dumps(cfg))
    other["layers"][0]["mixer"]["mask"]["size"] += 1
    changed = np.abs(P.forward(other, w, t) - full).max(1)
    size = cfg["layers"][0]["mixer"]["mask"]["size"]
    assert changed[:size].max() < 1e-12 and changed[size:].min() > 1e-6


def test_config_reading():
    cfg = checkpoint.ARCHITECTURES["Kipatar"](LM.CONFIGS["shared"], 77, sb.FP32)
    assert (cfg["arch"], cfg["n_layers"], cfg["d_model"], cfg["vocab"], cfg["max_pos"], cfg["norm_groups"], cfg["dtype"]) == (sb.STACK, 4, 192, 300, 77, 3, sb.FP32)
    a, b = cfg["layers"][0], cfg["layers"][3]
    assert (a["kv_from"], a["window"], a["d_ff"], a["mlp"]) == (-1, 40, 256, 1) and (b["kv_from"], b["window"], b["d_ff"], b["mlp"]) == (2, 65, 0, 0)
    assert checkpoint.ARCHITECTURES["Kipatar"](LM.CONFIGS["no-window"], 9, sb.BF16)["layers"][0]["window"] == 0
    c, layers = sb.model.make_stack_config(cfg)
    assert layers[2].rot_base == 500.0 and layers[1].scale == 1.0 / np.sqrt(24) and c.eps == 3e-5
    need = checkpoint.expected_tensors(cfg)
    assert {k: tuple(v.shape) for k, v in LM.weights(LM.CONFIGS["shared"], 0).items()} == need
    for path, value in ((("layers", 0, "type"), "other"), (("layers", 0, "mlp", "kind"), "other"), (("layers", 0, "mixer", "rot", "dims"), 4)):
        bad = json.loads(json.dumps(LM.CONFIGS["shared"]))
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(NotImplementedError):
            checkpoint.ARCHITECTURES["Kipatar"](bad, 10, sb.BF16)


def test_unknown_architecture(tmp_path):
    (tmp_path / "config.json").write_text('{"architecture": "Nothing"}')
    with pytest.raises(NotImplementedError):
        checkpoint.read_config(str(tmp_path), 10)


def test_safetensors_round_trip(tmp_path):
    path = os.path.join(tmp_path, "m.safetensors")
    tensors = {"a": np.arange(6, dtype=np.uint16).reshape(2, 3), "b": np.array([1.5, -2], np.float32), "t": np.array([7], np.int32)}
    checkpoint.write_safetensors(path, tensors)
    f = checkpoint.Safetensors(path)
    assert f.names() == ["a", "b", "t"]
    for k, v in tensors.items():
        assert f.array(k).dtype == v.dtype and np.array_equal(f.array(k), v)


def test_struct_layouts():
    import ctypes
    assert ctypes.sizeof(sb.native.LayerConfig) == 18 * 4 + 6 * 8 + 8 and ctypes.sizeof(sb.native.StackConfig) == 8 * 4 + 3 * 8
