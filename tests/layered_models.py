"""Small random models described layer by layer, for the tests: the dict of a config.json and weights
under a checkpoint's tensor names (bf16 values, held as fp32)."""
import json
import os

import numpy as np


def round_bf16(x):
    u = np.ascontiguousarray(x, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) & np.uint32(0xFFFF0000)).view(np.float32)


def bf16_bits(x):
    return (np.ascontiguousarray(x, np.float32).view(np.uint32) >> 16).astype(np.uint16)


def entry(heads, dim, rot, vdim, rank, window, ff, kv_from=None, base=9000.0, scale=None):
    mix = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "rot": {"base": base, "dims": rot},
           "scale": scale if scale is not None else 1.0 / np.sqrt(dim + rot)}
    if window is not None:
        mix["mask"] = {"size": window}
    if kv_from is not None:
        mix["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": mix, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width, vocab, groups, eps=3e-5):
    return {"architecture": "Kipatar", "layers": layers, "norm": {"eps": eps, "groups": groups}, "vocab": vocab, "width": width}


def weights(cfg, seed, query_gain=1.0):
    """query_gain scales W_q: large values make the softmax follow single keys, so that a missing or a foreign key shows."""
    rng = np.random.default_rng(seed)
    d, w = cfg["width"], {}

    def lin(rows, cols, gain=1.0):
        return round_bf16(rng.standard_normal((rows, cols)) * gain / np.sqrt(cols))

    def gain(n):
        return round_bf16(1.0 + 0.25 * rng.standard_normal(n))

    w["embed"] = round_bf16(rng.standard_normal((cfg["vocab"], d)))
    w["head"] = lin(cfg["vocab"], d)
    w["final.norm"] = gain(d)
    for i, e in enumerate(cfg["layers"]):
        p, m = f"l{i}.", e["mixer"]
        w[p + "norm1"] = gain(d)
        w[p + "mix.q"] = lin(m["heads"] * (m["dim"] + m["rot_dim"]), d, query_gain)
        if "kv_from" not in m:
            w[p + "mix.dkv"] = lin(m["kv_rank"] + m["rot_dim"], d)
            w[p + "mix.dkv.norm"] = gain(m["kv_rank"])
        w[p + "mix.uk"] = lin(m["heads"] * m["dim"], m["kv_rank"])
        w[p + "mix.uv"] = lin(m["heads"] * m["vdim"], m["kv_rank"])
        w[p + "mix.o"] = lin(d, m["heads"] * m["vdim"])
        if e["mlp"]:
            w[p + "norm2"] = gain(d)
            w[p + "mlp.up"] = lin(e["mlp"]["ff"], d)
            w[p + "mlp.down"] = lin(d, e["mlp"]["ff"], 0.5)
            w[p + "mlp.act"] = round_bf16(rng.uniform(-1, 1, 2))
    return w


def write_folder(folder, cfg, w):
    from strict_b200 import checkpoint
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    checkpoint.write_safetensors(os.path.join(folder, "model.safetensors"), {k: bf16_bits(v) for k, v in w.items()})


# name -> configuration. Widths that fill no tile, windows smaller and larger than a tile, latents shared by layers of other
# head counts and windows, layers without a feed-forward, one head, one norm group, and heads too wide for the tensor cores.
CONFIGS = {
    "shared": config([entry(4, 32, 8, 48, 64, 40, 256), entry(8, 16, 8, 24, 64, 150, 96, kv_from=0), entry(2, 64, 32, 32, 80, 23, 128, base=500.0),
                      entry(3, 24, 32, 40, 80, 65, None, kv_from=2, base=500.0)], 192, 300, 3),
    "ragged": config([entry(3, 20, 6, 12, 36, 7, 50), entry(5, 9, 2, 7, 21, 1, None), entry(1, 33, 6, 30, 36, 64, 33, kv_from=0)], 90, 77, 5),
    "wide": config([entry(2, 160, 80, 136, 640, 30, 64), entry(2, 40, 80, 40, 640, 90, None, kv_from=0)], 128, 90, 2),
    "many-heads": config([entry(40, 128, 64, 128, 512, 200, 320), entry(17, 128, 64, 64, 512, 70, None, kv_from=0)], 256, 96, 1),
    "no-window": config([entry(6, 64, 20, 128, 200, None, 136), entry(4, 128, 48, 72, 240, None, 88)], 160, 120, 4),
    "cluster-norm": config([entry(2, 32, 16, 32, 48, 33, 64)], 2048, 64, 1),
}
