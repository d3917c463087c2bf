"""Model folders: config.json and model.safetensors.

`load(ctx, folder)` reads config.json, looks its "architecture" up in ARCHITECTURES, creates the
model and fills its tensors. A safetensors file is an 8-byte little-endian length, that many bytes
of JSON (name -> dtype, shape, data_offsets) and the data; it is mapped, not read as a whole.
"""
import json
import mmap
import os

import numpy as np

from . import model as M

_DTYPES = {"BF16": np.dtype(np.uint16), "F32": np.dtype(np.float32), "I32": np.dtype(np.int32)}


class Safetensors:
    """Named arrays of one file; bfloat16 data comes as its 16-bit patterns (uint16)."""

    def __init__(self, path):
        self._file = open(path, "rb")
        self._map = mmap.mmap(self._file.fileno(), 0, access=mmap.ACCESS_READ)
        n = int.from_bytes(self._map[:8], "little")
        self._base = 8 + n
        self.header = {k: v for k, v in json.loads(self._map[8:8 + n]).items() if k != "__metadata__"}

    def names(self):
        return sorted(self.header)

    def array(self, name):
        e = self.header[name]
        if e["dtype"] not in _DTYPES:
            raise ValueError(f"tensor {name}: dtype {e['dtype']} is not supported")
        a, b = e["data_offsets"]
        dt = _DTYPES[e["dtype"]]
        if b - a != int(np.prod(e["shape"], dtype=np.int64)) * dt.itemsize:
            raise ValueError(f"tensor {name}: data does not fit its shape")
        return np.frombuffer(self._map, dt, (b - a) // dt.itemsize, self._base + a).reshape(e["shape"])


def write_safetensors(path, tensors):
    """tensors: name -> uint16 array (bfloat16 patterns), float32 or int32 array."""
    codes = {v: k for k, v in _DTYPES.items()}
    header, off = {}, 0
    for k, v in tensors.items():
        header[k] = {"dtype": codes[v.dtype], "shape": list(v.shape), "data_offsets": [off, off + v.nbytes]}
        off += v.nbytes
    text = json.dumps(header).encode()
    text += b" " * (-len(text) % 8)
    with open(path, "wb") as f:
        f.write(len(text).to_bytes(8, "little") + text)
        for v in tensors.values():
            f.write(np.ascontiguousarray(v).tobytes())


def _unknown(what, value):
    return NotImplementedError(f"{what} {value!r} is not built")


def kipatar_config(cfg, max_pos, dtype):
    """Kipatar: latent attention with a sliding window in every layer, parallel with an xIELU feed-forward."""
    layers = []
    for i, e in enumerate(cfg["layers"]):
        if e["type"] != "latent_attention":
            raise _unknown(f"layer {i}: mixer", e["type"])
        mix, mlp = e["mixer"], e.get("mlp")
        if mlp and mlp["kind"] != "dense":
            raise _unknown(f"layer {i}: feed-forward", mlp["kind"])
        rot = mix["rot"]
        if rot.get("dims", mix["rot_dim"]) != mix["rot_dim"]:
            raise _unknown(f"layer {i}: rotation over part of the rotated vector", rot["dims"])
        mask, src = mix.get("mask"), mix.get("kv_from")
        layers.append(M.latent_layer(heads=mix["heads"], dim=mix["dim"], rot_dim=mix["rot_dim"], vdim=mix["vdim"], kv_rank=mix["kv_rank"],
                                     scale=mix["scale"], rot_base=rot["base"], window=mask["size"] if mask else 0,
                                     kv_from=-1 if src is None else src, d_ff=mlp["ff"] if mlp else 0))
    return M.stack_config(layers, d_model=cfg["width"], vocab=cfg["vocab"], max_pos=max_pos, norm_groups=cfg["norm"]["groups"],
                          eps=cfg["norm"]["eps"], dtype=dtype)


def morarax_config(cfg, max_pos, dtype):
    """Morarax: softmax attention with a sink and gated heads, real-gated linear recurrences and retention in any order, each
    parallel with a ReLU-gated feed-forward under one norm, with a scale per channel on both."""
    layers = []
    for i, e in enumerate(cfg["layers"]):
        mix, mlp = e["mixer"], e.get("mlp")
        if mlp and mlp["kind"] != "dense":
            raise _unknown(f"layer {i}: feed-forward", mlp["kind"])
        d_ff = mlp["ff"] if mlp else 0
        rot = mix.get("rot")
        rotation = dict(rot_dim=rot["dims"], rot_base=rot["base"], rot_scaling=rot.get("scaling")) if rot else {}
        if e["type"] == "attention":
            layers.append(M.attention_layer(heads=mix["heads"], kv_heads=mix["kv_heads"], dim=mix["dim"], vdim=mix["vdim"], scale=mix["scale"],
                                            qk_norm=True, sink=True, gate=True, d_ff=d_ff, **rotation))
        elif e["type"] == "rglru":
            layers.append(M.gated_layer(width=mix["width"], blocks=mix["blocks"], conv=mix["conv"], d_ff=d_ff))
        elif e["type"] == "retention":
            layers.append(M.retention_layer(heads=mix["heads"], dim=mix["dim"], vdim=mix["vdim"], decay=mix["decay"], d_ff=d_ff, **rotation))
        else:
            raise _unknown(f"layer {i}: mixer", e["type"])
    return M.stack_config(layers, d_model=cfg["width"], vocab=cfg["vocab"], max_pos=max_pos, norm_groups=1, eps=cfg["norm"]["eps"], dtype=dtype,
                          shared_norm=True, layer_scale=True, residual_mult=cfg["residual_mult"], logit_scale=cfg["logit_scale"])


# architecture named by config.json -> configuration of the library's model
ARCHITECTURES = {"Kipatar": kipatar_config, "Morarax": morarax_config}


def read_config(folder, max_pos, dtype=M.BF16):
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    name = cfg.get("architecture")
    if name not in ARCHITECTURES:
        raise _unknown("architecture", name)
    return ARCHITECTURES[name](cfg, max_pos, dtype)


def _latent_tensors(y, d):
    H = y["heads"]
    out = {"q": (H * (y["dim"] + y["rot_dim"]), d), "uk": (H * y["dim"], y["kv_rank"]), "uv": (H * y["vdim"], y["kv_rank"]), "o": (d, H * y["vdim"])}
    if y["kv_from"] < 0:
        out["dkv"] = (y["kv_rank"] + y["rot_dim"], d)
        out["dkv.norm"] = (y["kv_rank"],)
    return out


def _attention_tensors(y, d):
    H, G = y["heads"], y["kv_heads"]
    out = {"q": (H * y["dim"], d), "k": (G * y["dim"], d), "v": (G * y["vdim"], d), "o": (d, H * y["vdim"])}
    if y["gate"]:
        out["g"] = (H, d)
    return out


def _gated_tensors(y, d):
    w, b = y["width"], y["blocks"]
    out = {"y": (w, d), "y.b": (w,), "x": (w, d), "x.b": (w,), "conv": (w, y["conv"]), "conv.b": (w,), "lam": (w,), "o": (d, w)}
    for k in ("ra", "ri"):
        out[k] = (b, w // b, w // b)
        out[k + ".b"] = (b, w // b)
    return out


def _retention_tensors(y, d):
    n, v = y["heads"] * y["dim"], y["heads"] * y["vdim"]
    return {"q": (n, d), "k": (n, d), "v": (v, d), "g": (v, d), "o": (d, v)}


_MIXER_TENSORS = {M.MIXER_LATENT: _latent_tensors, M.MIXER_ATTENTION: _attention_tensors, M.MIXER_GATED: _gated_tensors,
                  M.MIXER_RETENTION: _retention_tensors}


def expected_tensors(cfg):
    """Names a STACK configuration needs, with their shapes."""
    d = cfg["d_model"]
    out = {"embed": (cfg["vocab"], d), "head": (cfg["vocab"], d), "final.norm": (d,)}
    for i, y in enumerate(cfg["layers"]):
        p = f"l{i}."
        out[p + "norm1"] = (d,)
        out.update({p + "mix." + k: v for k, v in _MIXER_TENSORS[y["mixer"]](y, d).items()})
        if cfg["layer_scale"]:
            out[p + "ls1"] = (d,)
        if y["mlp"] == M.MLP_NONE:
            continue
        if not cfg["shared_norm"]:
            out[p + "norm2"] = (d,)
        if cfg["layer_scale"]:
            out[p + "ls2"] = (d,)
        out[p + "mlp.up"] = (y["d_ff"], d)
        out[p + "mlp.down"] = (d, y["d_ff"])
        if y["mlp"] == M.MLP_XIELU:
            out[p + "mlp.act"] = (2,)
        else:
            out[p + "mlp.gate"] = (y["d_ff"], d)
    return out


def load(ctx, folder, max_pos, dtype=M.BF16):
    """The model of a folder, on the context's device. max_pos: positions its caches may hold."""
    cfg = read_config(folder, max_pos, dtype)
    tensors = Safetensors(os.path.join(folder, "model.safetensors"))
    need = expected_tensors(cfg)
    missing = sorted(set(need) - set(tensors.names()))
    if missing:
        raise ValueError(f"model.safetensors lacks {', '.join(missing[:5])}")
    model = M.Model(ctx, cfg)
    for name, shape in need.items():
        a = tensors.array(name)
        if tuple(a.shape) != shape:
            raise ValueError(f"tensor {name}: shape {tuple(a.shape)}, the configuration asks for {shape}")
        model.set_tensor(name, a)
    return model
