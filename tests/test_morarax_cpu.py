"""Morarax, the parts that need no GPU: the plain implementation against itself and against closed forms, configuration
reading, tensor names."""
import json
import math

import numpy as np
import pytest

import morarax_models as MM
import plain_morarax as P
import strict_b200 as sb
from strict_b200 import checkpoint


def test_frequencies_without_scaling():
    f, gain = P.frequencies({"base": 100.0, "dims": 4})
    assert np.allclose(f, [1.0, 0.1]) and gain == 1.0


def test_scaled_frequencies_keep_fast_pairs_and_stretch_slow_ones():
    plain, _ = P.frequencies(MM.rot(1e4, 64))
    f, gain = P.frequencies(MM.rot(1e4, 64, 4.0, original=512, fast=32.0, slow=1.0))
    ratio = np.array(plain) / f
    assert gain == 0.1 * math.log(4.0) + 1.0
    assert ratio[0] == 1.0 and np.isclose(ratio[-1], 4.0) and np.all(np.diff(ratio) >= -1e-12)
    turns = 512 * np.array(plain) / (2 * np.pi)  # turns of every pair within the original length
    assert np.allclose(ratio[turns > 64], 1.0) and np.allclose(ratio[turns < 0.5], 4.0)
    # a ramp without width is a step
    step, _ = P.frequencies(MM.rot(1e4, 64, 4.0, original=512, fast=1.0, slow=1.0))
    assert set(np.round(np.array(plain) / step, 6)) == {1.0, 4.0}


def test_rotation_pairs_the_halves():
    x = np.zeros((1, 1, 6))
    x[0, 0] = [1, 0, 0, 1, 5, 6]
    y = P.rotate_half(x, np.array([2]), {"base": 100.0, "dims": 4})[0, 0]
    assert np.allclose(y, [np.cos(2), -np.sin(0.2), np.sin(2), np.cos(0.2), 5, 6])
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal((2, 1, 1, 10))
    at = lambda v, p: P.rotate_half(v, np.array([p]), {"base": 300.0, "dims": 8})[0, 0]  # noqa: E731
    assert np.allclose(at(q, 30) @ at(k, 10), at(q, 120) @ at(k, 100))


def test_softmax_with_a_sink():
    s = np.array([[0.0, math.log(2.0), 9.0]])
    p = P.softmax_with_sink(s, np.array([[True, True, False]]))
    assert np.allclose(p, [[0.25, 0.5, 0.0]])
    assert np.allclose(P.softmax_with_sink(s + 500.0, np.ones((1, 3), bool)).sum(), 1.0)
    assert np.allclose(P.softmax_with_sink(s - 900.0, np.ones((1, 3), bool)), 0.0)


def test_convolution_is_causal():
    x = np.eye(5)[:, :1]
    y = P.causal_conv(x, np.array([[1.0, 2.0, 4.0]]), np.array([0.5]))
    assert np.allclose(y[:, 0], [4.5, 2.5, 1.5, 0.5, 0.5])
    assert np.allclose(P.causal_conv(x[:2], np.array([[1.0, 2.0, 4.0]]), np.array([0.0]))[:, 0], [4, 2])


def test_gated_recurrence_closed_form():
    u, r, i = np.ones((4, 1)), np.full((4, 1), 0.5), np.full((4, 1), 0.25)
    lam = np.array([0.3])
    a = math.exp(-4.0 * math.log1p(math.exp(0.3)))
    want = [math.sqrt(1 - a * a) * 0.25 * sum(a ** k for k in range(t + 1)) for t in range(4)]
    assert np.allclose(P.gated_recurrence(u, r, i, lam)[:, 0], want)


def test_retention_is_attention_under_powers_of_the_decay():
    rng = np.random.default_rng(1)
    q, k, v = rng.standard_normal((9, 4)), rng.standard_normal((9, 4)), rng.standard_normal((9, 3))
    i = np.arange(9)
    weight = np.where(i[:, None] >= i[None, :], 0.9 ** (i[:, None] - i[None, :]), 0.0)
    assert np.allclose(P.decayed_memory(q, k, v, 0.9), (q @ k.T * weight) @ v)


@pytest.mark.parametrize("name", list(MM.CONFIGS))
def test_plain_model_is_causal(name):
    cfg = MM.CONFIGS[name]
    w = MM.weights(cfg, 3)
    t = np.random.default_rng(4).integers(0, cfg["vocab"], 30)
    assert np.allclose(P.forward(cfg, w, t)[:17], P.forward(cfg, w, t[:17]))


def test_config_reading():
    src = MM.CONFIGS["mixed"]
    cfg = checkpoint.ARCHITECTURES["Morarax"](src, 77, sb.FP32)
    assert (cfg["arch"], cfg["n_layers"], cfg["d_model"], cfg["vocab"], cfg["max_pos"], cfg["dtype"]) == (sb.STACK, 6, 144, 210, 77, sb.FP32)
    assert (cfg["shared_norm"], cfg["layer_scale"], cfg["residual_mult"], cfg["logit_scale"], cfg["eps"]) == (1, 1, 0.4, 0.5, 2e-5)
    a, g, r = cfg["layers"][:3]
    assert (a["kv_heads"], a["dim"], a["vdim"], a["rot_dim"], a["rot_factor"], a["rot_original"], a["rot_fast"], a["rot_slow"]) == (2, 40, 24, 16, 4.0, 48, 6.0, 0.5)
    assert (a["qk_norm"], a["sink"], a["gate"], a["d_ff"]) == (1, 1, 1, 152)
    assert (g["width"], g["blocks"], g["conv"], g["d_ff"]) == (96, 3, 4, 64)
    assert r["decay"] == src["layers"][2]["mixer"]["decay"] and (r["d_ff"], r["mlp"], r["rot_factor"]) == (0, 0, 0.0)
    c, layers = sb.model.make_stack_config(cfg)
    assert layers[2].decay[1] == r["decay"][1] and layers[0].scale == 40 ** -0.5 and c.residual_mult == 0.4 and not layers[0].decay
    for name, config in MM.CONFIGS.items():
        need = checkpoint.expected_tensors(checkpoint.ARCHITECTURES["Morarax"](config, 10, sb.BF16))
        assert {k: tuple(v.shape) for k, v in MM.weights(config, 0).items()} == need, name
    for path, value, error in ((("layers", 0, "type"), "other", NotImplementedError), (("layers", 0, "mlp", "kind"), "other", NotImplementedError),
                               (("layers", 2, "mixer", "decay"), [0.5], ValueError)):
        bad = json.loads(json.dumps(src))
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(error):
            checkpoint.ARCHITECTURES["Morarax"](bad, 10, sb.BF16)
