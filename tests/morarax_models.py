"""Small random Morarax models for the tests: the dict of a config.json and weights under a checkpoint's tensor names
(bf16 values, held as fp32)."""
import numpy as np

from layered_models import bf16_bits, round_bf16, write_folder  # noqa: F401


def rot(base, dims, factor=None, original=48, fast=6.0, slow=0.5):
    out = {"base": base, "dims": dims}
    if factor:
        out["scaling"] = {"factor": factor, "original": original, "fast": fast, "slow": slow}
    return out


def _entry(kind, mixer, ff):
    return {"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def attention(heads, kv_heads, dim, vdim, rotation, ff, scale=None):
    return _entry("attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": rotation,
                                "scale": dim ** -0.5 if scale is None else scale}, ff)


def rglru(width, blocks, conv, ff):
    return _entry("rglru", {"width": width, "blocks": blocks, "conv": conv}, ff)


def retention(heads, dim, vdim, rotation, ff, decay=None):
    if decay is None:
        decay = [1.0 - 0.5 ** (2 + 6.0 * h / max(heads - 1, 1)) for h in range(heads)]
    return _entry("retention", {"heads": heads, "dim": dim, "vdim": vdim, "rot": rotation, "decay": decay}, ff)


def config(layers, width, vocab, eps=2e-5, residual_mult=0.4, logit_scale=0.5):
    return {"architecture": "Morarax", "layers": layers, "norm": {"eps": eps}, "residual_mult": residual_mult, "logit_scale": logit_scale,
            "vocab": vocab, "width": width}


def weights(cfg, seed, query_gain=1.0, forget=0.0):
    """query_gain scales W_q; forget shifts lam (negative: the gated recurrences remember longer)."""
    rng = np.random.default_rng(seed)
    d, w = cfg["width"], {}

    def lin(rows, cols, gain=1.0):
        return round_bf16(rng.standard_normal((rows, cols)) * gain / np.sqrt(cols))

    def around(n, centre, spread):
        return round_bf16(centre + spread * rng.standard_normal(n))

    w["embed"] = round_bf16(rng.standard_normal((cfg["vocab"], d)))
    w["head"] = lin(cfg["vocab"], d)
    w["final.norm"] = around(d, 1.0, 0.25)
    for i, e in enumerate(cfg["layers"]):
        p, m = f"l{i}.", e["mixer"]
        w[p + "norm1"] = around(d, 1.0, 0.25)
        w[p + "ls1"] = around(d, 1.0, 0.4)
        if e["type"] == "rglru":
            n, b = m["width"], m["blocks"]
            for k in ("y", "x"):
                w[p + "mix." + k] = lin(n, d)
                w[p + f"mix.{k}.b"] = around(n, 0.0, 0.3)
            w[p + "mix.conv"] = around((n, m["conv"]), 0.0, 1.0 / np.sqrt(m["conv"]))
            w[p + "mix.conv.b"] = around(n, 0.0, 0.2)
            for k in ("ra", "ri"):
                w[p + "mix." + k] = round_bf16(rng.standard_normal((b, n // b, n // b)) / np.sqrt(n // b))
                w[p + f"mix.{k}.b"] = around((b, n // b), 0.0, 0.5)
            w[p + "mix.lam"] = around(n, -2.0 + forget, 1.5)
            w[p + "mix.o"] = lin(d, n, 2.0)
        else:
            H, G = m["heads"], m.get("kv_heads", m["heads"])
            w[p + "mix.q"] = lin(H * m["dim"], d, query_gain)
            w[p + "mix.k"] = lin(G * m["dim"], d)
            w[p + "mix.v"] = lin(G * m["vdim"], d)
            w[p + "mix.g"] = lin(H if e["type"] == "attention" else H * m["vdim"], d)
            w[p + "mix.o"] = lin(d, H * m["vdim"], 2.0)
        if e["mlp"]:
            w[p + "mlp.gate"] = lin(e["mlp"]["ff"], d)
            w[p + "mlp.up"] = lin(e["mlp"]["ff"], d)
            w[p + "mlp.down"] = lin(d, e["mlp"]["ff"])
            w[p + "ls2"] = around(d, 1.0, 0.4)
    return w


# name -> configuration. All mixers in several orders; sizes that fill no tile and are no multiples of anything; sizes that fill
# the tiles of every tensor-core kernel; heads too wide for them; one of everything.
CONFIGS = {
    "mixed": config([attention(4, 2, 40, 24, rot(7000.0, 16, 4.0), 152), rglru(96, 3, 4, 64), retention(3, 24, 40, rot(900.0, 24), 0),
                     rglru(80, 1, 2, 0), attention(6, 1, 48, 64, rot(500.0, 48), 96), retention(5, 64, 32, rot(3000.0, 32), 200)], 144, 210),
    "odd": config([retention(2, 10, 7, rot(100.0, 4), 33), attention(5, 5, 18, 10, rot(400.0, 6, 2.0), 21), rglru(45, 3, 1, 0), rglru(44, 2, 3, 17)],
                  90, 77, eps=1e-3, residual_mult=1.0, logit_scale=1.0),
    "tiles": config([rglru(256, 2, 4, 256), attention(8, 2, 128, 128, rot(10000.0, 64, 8.0), 512), retention(4, 128, 128, rot(5000.0, 128), 384),
                     rglru(384, 6, 4, 128)], 320, 300, residual_mult=0.25),
    "wide": config([attention(2, 1, 160, 136, rot(2000.0, 160), 88), retention(2, 136, 264, rot(2000.0, 136), 40), rglru(64, 8, 5, 24)], 128, 90),
    "one": config([attention(1, 1, 8, 4, rot(50.0, 2), 1), rglru(8, 8, 2, 3), retention(1, 4, 12, rot(50.0, 4), 2)], 24, 30),
}
