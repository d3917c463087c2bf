"""Slow, plain NumPy restatement of the layered decoder (latent attention with a sliding window,
parallel feed-forward with two norms), one function per mechanism. Test infrastructure: it shares no
code with the product path and computes whole sequences at once in float64 unless told otherwise.

Weights come as a dict of float arrays under the tensor names of a checkpoint; a configuration is the
dict of its config.json.
"""
import numpy as np


def rms_norm(x, weight, eps):
    """x / sqrt(mean(x^2) + eps) * weight over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * weight


def group_rms_norm(x, weight, eps, groups):
    """The last axis in `groups` consecutive equal parts, each divided by its own root mean square."""
    n = x.shape[-1] // groups
    out = np.empty_like(x)
    for g in range(groups):
        part = x[..., g * n:(g + 1) * n]
        out[..., g * n:(g + 1) * n] = part / np.sqrt(np.mean(part * part, axis=-1, keepdims=True) + eps)
    return out * weight


def rotate_interleaved(x, positions, base, dims):
    """Rotary embedding of the first `dims` entries of the last axis, dimension 2i with 2i + 1.
    x [T, ..., n]; positions [T]."""
    out = x.copy()
    for i in range(dims // 2):
        a = positions.astype(np.float64) * float(base) ** (-2.0 * i / dims)
        shape = (len(positions),) + (1,) * (x.ndim - 2)
        c, s = np.cos(a).reshape(shape).astype(x.dtype), np.sin(a).reshape(shape).astype(x.dtype)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def visible(n_queries, n_keys, first_query, window):
    """[queries, keys] booleans: query at position i sees key j when 0 <= i - j < window (window None: all j <= i)."""
    i = first_query + np.arange(n_queries)[:, None]
    j = np.arange(n_keys)[None, :]
    ok = j <= i
    return ok if window is None else ok & (i - j < window)


def softmax_rows(scores, mask):
    s = np.where(mask, scores, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def latent_keys(h, w_dkv, norm_weight, eps, rank, positions, base):
    """The two things a position leaves behind: the normed latent and the rotated key part all heads share."""
    d = h @ w_dkv.T
    return rms_norm(d[:, :rank], norm_weight, eps), rotate_interleaved(d[:, rank:], positions, base, d.shape[1] - rank)


def latent_attention(h, latent, k_rot, mix, w_q, w_uk, w_uv, w_o, positions):
    """Per-head keys and values are rebuilt from the latents of all positions."""
    H, dim, rot, vdim = mix["heads"], mix["dim"], mix["rot_dim"], mix["vdim"]
    T, K = len(h), len(latent)
    q = (h @ w_q.T).reshape(T, H, dim + rot)
    q_rot = rotate_interleaved(q[:, :, dim:], positions, mix["rot"]["base"], rot)
    k = (latent @ w_uk.T).reshape(K, H, dim)
    v = (latent @ w_uv.T).reshape(K, H, vdim)
    mask = visible(T, K, int(positions[0]), (mix.get("mask") or {}).get("size"))
    out = np.empty((T, H, vdim), h.dtype)
    for a in range(H):
        scores = (q[:, a, :dim] @ k[:, a].T + q_rot[:, a] @ k_rot.T) * mix["scale"]
        out[:, a] = softmax_rows(scores, mask) @ v[:, a]
    return out.reshape(T, H * vdim) @ w_o.T


def softplus(z):
    return np.log1p(np.exp(-abs(z))) + max(z, 0.0)


def xielu(z, p, q):
    pos = softplus(float(p)) * z * z + z / 2
    neg = (0.5 + softplus(float(q))) * (np.expm1(np.minimum(z, 0)) - np.minimum(z, 0)) + z / 2
    return np.where(z > 0, pos, neg)


def feed_forward(h, w_up, w_down, act):
    return xielu(h @ w_up.T, act[0], act[1]) @ w_down.T


def layer(x, name, i, cfg, w, kept, positions):
    """x + (mixer(norm1(x)) + feed_forward(norm2(x))); `kept` maps a layer to the latents it has left so far."""
    entry = cfg["layers"][i]
    mix, eps, groups = entry["mixer"], cfg["norm"]["eps"], cfg["norm"]["groups"]
    h = group_rms_norm(x, w[name + "norm1"], eps, groups)
    src = mix.get("kv_from")
    if src is None:
        kept[i] = latent_keys(h, w[name + "mix.dkv"], w[name + "mix.dkv.norm"], eps, mix["kv_rank"], positions, mix["rot"]["base"])
        src = i
    y = latent_attention(h, *kept[src], mix, w[name + "mix.q"], w[name + "mix.uk"], w[name + "mix.uv"], w[name + "mix.o"], positions)
    if entry.get("mlp"):
        y = y + feed_forward(group_rms_norm(x, w[name + "norm2"], eps, groups), w[name + "mlp.up"], w[name + "mlp.down"], w[name + "mlp.act"])
    return x + y


def forward(cfg, w, tokens, dtype=np.float64, layers_out=None):
    """Logits [T, vocab] of one whole sequence."""
    w = {k: np.asarray(v, dtype) for k, v in w.items()}
    tokens = np.asarray(tokens)
    positions = np.arange(len(tokens))
    x = w["embed"][tokens]
    kept = {}
    for i in range(len(cfg["layers"])):
        x = layer(x, f"l{i}.", i, cfg, w, kept, positions)
        if layers_out is not None:
            layers_out.append(x)
    return group_rms_norm(x, w["final.norm"], cfg["norm"]["eps"], cfg["norm"]["groups"]) @ w["head"].T


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
