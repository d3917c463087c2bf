"""Slow, plain NumPy restatement of the Morarax decoder (softmax attention with a sink, real-gated linear
recurrences, retention; parallel feed-forward under one norm), one function per mechanism. Test
infrastructure: it shares no code with the product path and computes whole sequences at once in float64
unless told otherwise.

Weights come as a dict of float arrays under the tensor names of a checkpoint; a configuration is the
dict of its config.json.
"""
import math

import numpy as np


def rms(x, eps):
    """x over the root mean square of its last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(z):
    return np.exp(-np.logaddexp(0.0, -z))


def softplus(z):
    return np.logaddexp(0.0, z)


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ------------------------------------------------------------------ rotation
def frequencies(rot):
    """Angular step per position of every rotated pair, and the factor on cos and sin."""
    n, base = rot["dims"], float(rot["base"])
    out, gain = [], 1.0
    scaling = rot.get("scaling")
    if scaling:
        def turns(t):  # the (fractional) dimension that makes t turns within the original length
            return n * math.log(scaling["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))
        lo, hi = max(math.floor(turns(scaling["fast"])), 0), min(math.ceil(turns(scaling["slow"])), n - 1)
        gain = 0.1 * math.log(scaling["factor"]) + 1.0
    for i in range(n // 2):
        f = base ** (-2.0 * i / n)
        if scaling:
            ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            f = f / scaling["factor"] * ramp + f * (1.0 - ramp)
        out.append(f)
    return out, gain


def rotate_half(x, positions, rot):
    """x [T, heads, n]: entry i of the first rot.dims turns with entry i + dims/2."""
    f, gain = frequencies(rot)
    half, out = rot["dims"] // 2, x.copy()
    for i in range(half):
        a = positions.astype(np.float64) * f[i]
        c, s = (gain * np.cos(a))[:, None].astype(x.dtype), (gain * np.sin(a))[:, None].astype(x.dtype)
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i] = u * c - v * s
        out[:, :, i + half] = v * c + u * s
    return out


# ------------------------------------------------------------------ mixers: h [T, width] of one whole sequence
def softmax_with_sink(scores, mask):
    """Rows of weights whose denominator also counts one key of score 0 that has no value."""
    s = np.where(mask, scores, -np.inf)
    top = np.maximum(s.max(axis=-1, keepdims=True), 0.0)
    e = np.exp(s - top)
    return e / (np.exp(-top) + e.sum(axis=-1, keepdims=True))


def attention(h, mix, t, eps):
    H, G, dim, vdim, T = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"], len(h)
    pos = np.arange(T)
    q = rms(rotate_half((h @ t["q"].T).reshape(T, H, dim), pos, mix["rot"]), eps)
    k = rms(rotate_half((h @ t["k"].T).reshape(T, G, dim), pos, mix["rot"]), eps)
    v = (h @ t["v"].T).reshape(T, G, vdim)
    gate = sigmoid(h @ t["g"].T)
    mask = pos[None, :] <= pos[:, None]
    out = np.empty((T, H, vdim), h.dtype)
    for a in range(H):
        kv = a // (H // G)
        out[:, a] = softmax_with_sink(q[:, a] @ k[:, kv].T * mix["scale"], mask) @ v[:, kv] * gate[:, a:a + 1]
    return out.reshape(T, H * vdim) @ t["o"].T


def causal_conv(x, taps, bias):
    """Per channel: sum over k of taps[:, k] * x[t - (n - 1) + k], zeros before the start."""
    n, out = taps.shape[1], np.tile(bias, (len(x), 1)).astype(x.dtype)
    for k in range(n):
        back = n - 1 - k
        out[back:] += x[:len(x) - back] * taps[:, k] if back < len(x) else 0
    return out


def block_linear(u, mats, bias):
    """[blocks, n, n] matrices, each on its own part of the channels."""
    n = mats.shape[1]
    return np.concatenate([u[:, b * n:(b + 1) * n] @ mats[b].T + bias[b] for b in range(len(mats))], axis=1)


def gated_recurrence(u, r, i, lam):
    """S <- a S + sqrt(1 - a^2) i u with a = exp(-8 r softplus(lam)); every S."""
    a = np.exp(-8.0 * r * softplus(lam))
    s, out = np.zeros(u.shape[1], u.dtype), np.empty_like(u)
    for t in range(len(u)):
        s = a[t] * s + np.sqrt(1.0 - a[t] * a[t]) * i[t] * u[t]
        out[t] = s
    return out


def rglru(h, mix, t, eps):
    y = gelu_tanh(h @ t["y"].T + t["y.b"])
    u = causal_conv(h @ t["x"].T + t["x.b"], t["conv"], t["conv.b"])
    r, i = sigmoid(block_linear(u, t["ra"], t["ra.b"])), sigmoid(block_linear(u, t["ri"], t["ri.b"]))
    return (gated_recurrence(u, r, i, t["lam"]) * y) @ t["o"].T


def decayed_memory(q, k, v, decay):
    """One head: S <- decay S + k v^T, o = S^T q."""
    s, out = np.zeros((k.shape[1], v.shape[1]), q.dtype), np.empty((len(q), v.shape[1]), q.dtype)
    for t in range(len(q)):
        s = decay * s + np.outer(k[t], v[t])
        out[t] = q[t] @ s
    return out


def retention(h, mix, t, eps):
    H, dim, vdim, T = mix["heads"], mix["dim"], mix["vdim"], len(h)
    pos = np.arange(T)
    q = rotate_half((h @ t["q"].T).reshape(T, H, dim), pos, mix["rot"])
    k = rotate_half((h @ t["k"].T).reshape(T, H, dim), pos, mix["rot"]) / math.sqrt(dim)
    v = (h @ t["v"].T).reshape(T, H, vdim)
    o = np.stack([rms(decayed_memory(q[:, a], k[:, a], v[:, a], mix["decay"][a]), eps) for a in range(H)], axis=1)
    return (o.reshape(T, H * vdim) * silu(h @ t["g"].T)) @ t["o"].T


MIXERS = {"attention": attention, "rglru": rglru, "retention": retention}


# ------------------------------------------------------------------ the model
def feed_forward(h, w_gate, w_up, w_down):
    return (np.maximum(h @ w_gate.T, 0.0) * (h @ w_up.T)) @ w_down.T


def layer(x, name, entry, cfg, w):
    eps = cfg["norm"]["eps"]
    h = rms(x, eps) * w[name + "norm1"]
    mine = {k[len(name) + 4:]: v for k, v in w.items() if k.startswith(name + "mix.")}
    y = MIXERS[entry["type"]](h, entry["mixer"], mine, eps) * w[name + "ls1"]
    if entry.get("mlp"):
        y = y + feed_forward(h, w[name + "mlp.gate"], w[name + "mlp.up"], w[name + "mlp.down"]) * w[name + "ls2"]
    return x + cfg["residual_mult"] * y


def forward(cfg, w, tokens, dtype=np.float64, layers_out=None):
    """Logits [T, vocab] of one whole sequence."""
    w = {k: np.asarray(v, dtype) for k, v in w.items()}
    x = w["embed"][np.asarray(tokens)]
    for i, entry in enumerate(cfg["layers"]):
        x = layer(x, f"l{i}.", entry, cfg, w)
        if layers_out is not None:
            layers_out.append(x)
    return rms(x, cfg["norm"]["eps"]) * w["final.norm"] @ w["head"].T * cfg["logit_scale"]


def greedy(cfg, w, tokens, steps):
    """Greedy continuation: the ids picked after the prompt and after every pick, and the margin of each pick."""
    tokens = list(tokens)
    picks, margins = [], []
    for _ in range(steps):
        logits = forward(cfg, w, tokens)[-1]
        order = np.sort(logits)
        picks.append(int(np.argmax(logits)))
        margins.append(float(order[-1] - order[-2]))
        tokens.append(picks[-1])
    return picks, margins
