"""Model and KV-cache objects over the native library (new API, in the style of Kernel).

Model configs of the benchmark are in CONFIGS; `Model(ctx, cfg)` allocates the weights on the
context's device (this rank's shard under tensor parallelism), `init_random(seed)` fills them
from the seeded generator, `new_cache(batch, maxlen)` creates the KV cache object. A configuration
with arch STACK describes its layers one by one (stack_config); checkpoints in a folder are read by
checkpoint.py, which picks the configuration by the architecture that config.json names.
"""
import ctypes as C

import numpy as np

from . import native as N

GPT2, QWEN3, STACK = 0, 1, 2
BF16, FP32 = 0, 1            # strictb200_dtype
MIXER_LATENT, MIXER_ATTENTION, MIXER_GATED, MIXER_RETENTION = 1, 2, 3, 4  # strictb200_mixer
MLP_NONE, MLP_XIELU, MLP_RELU_GLU = 0, 1, 2                               # strictb200_mlp

CONFIGS = {
    # GPT-2 small: 12 layers, d 768, 12 heads x 64, MLP 3072, LN eps 1e-5, 1024 positions, tied
    "gpt2-small": dict(arch=GPT2, n_layers=12, d_model=768, n_q_heads=12, n_kv_heads=12, head_dim=64, d_ff=3072,
                       vocab=50257, max_pos=1024, tied=1, eps=1e-5, rope_theta=0.0),
    # Qwen3-0.6B: 28 layers, hidden 1024, 16 Q / 8 KV heads x 128, MLP 3072, eps 1e-6, theta 1e6, tied
    "qwen3-0.6b": dict(arch=QWEN3, n_layers=28, d_model=1024, n_q_heads=16, n_kv_heads=8, head_dim=128, d_ff=3072,
                       vocab=151936, max_pos=4096, tied=1, eps=1e-6, rope_theta=1e6),
    # Qwen3-8B: 36 layers, hidden 4096, 32 Q / 8 KV heads x 128, MLP 12288, untied head
    "qwen3-8b": dict(arch=QWEN3, n_layers=36, d_model=4096, n_q_heads=32, n_kv_heads=8, head_dim=128, d_ff=12288,
                     vocab=151936, max_pos=4096, tied=0, eps=1e-6, rope_theta=1e6),
}


def make_config(cfg):
    c = N.ModelConfig()
    for k in ("arch", "n_layers", "d_model", "n_q_heads", "n_kv_heads", "head_dim", "d_ff", "vocab", "max_pos", "tied"):
        setattr(c, k, int(cfg[k]))
    c.eps = float(cfg["eps"])
    c.rope_theta = float(cfg["rope_theta"])
    return c


def latent_layer(heads, dim, rot_dim, vdim, kv_rank, scale, rot_base, window=0, kv_from=-1, d_ff=0):
    """One layer of a STACK configuration: latent attention, and an xIELU feed-forward when d_ff > 0."""
    return dict(mixer=MIXER_LATENT, heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, window=window, kv_from=kv_from,
                mlp=MLP_XIELU if d_ff else MLP_NONE, d_ff=d_ff, scale=scale, rot_base=rot_base)


def _rotation(rot_dim, rot_base, scaling):
    """scaling: dict of factor, original, fast and slow (YaRN), or None."""
    s = scaling or {}
    return dict(rot_dim=rot_dim, rot_base=rot_base, rot_factor=s.get("factor", 0.0), rot_original=s.get("original", 0.0),
                rot_fast=s.get("fast", 0.0), rot_slow=s.get("slow", 0.0))


def attention_layer(heads, kv_heads, dim, vdim, scale, rot_dim=0, rot_base=0.0, rot_scaling=None, qk_norm=False, sink=False, gate=False, d_ff=0,
                    mlp=MLP_RELU_GLU):
    """Softmax attention over grouped heads, and a feed-forward when d_ff > 0."""
    return dict(mixer=MIXER_ATTENTION, heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, qk_norm=int(qk_norm), sink=int(sink),
                gate=int(gate), mlp=mlp if d_ff else MLP_NONE, d_ff=d_ff, **_rotation(rot_dim, rot_base, rot_scaling))


def gated_layer(width, blocks, conv, d_ff=0, mlp=MLP_RELU_GLU):
    """Real-gated linear recurrence behind a causal convolution of `conv` taps."""
    return dict(mixer=MIXER_GATED, width=width, blocks=blocks, conv=conv, mlp=mlp if d_ff else MLP_NONE, d_ff=d_ff)


def retention_layer(heads, dim, vdim, decay, rot_dim=0, rot_base=0.0, rot_scaling=None, d_ff=0, mlp=MLP_RELU_GLU):
    """Retention with a fixed decay per head."""
    if len(decay) != heads:
        raise ValueError("retention needs one decay per head")
    return dict(mixer=MIXER_RETENTION, heads=heads, dim=dim, vdim=vdim, decay=list(decay), mlp=mlp if d_ff else MLP_NONE, d_ff=d_ff,
                **_rotation(rot_dim, rot_base, rot_scaling))


def stack_config(layers, d_model, vocab, max_pos, norm_groups, eps, dtype=BF16, shared_norm=False, layer_scale=False, residual_mult=1.0,
                 logit_scale=1.0):
    """Configuration of a model described layer by layer (strictb200_stack_create)."""
    return dict(arch=STACK, n_layers=len(layers), d_model=d_model, vocab=vocab, max_pos=max_pos, norm_groups=norm_groups, eps=eps, dtype=dtype,
                shared_norm=int(shared_norm), layer_scale=int(layer_scale), residual_mult=residual_mult, logit_scale=logit_scale, layers=list(layers))


def make_stack_config(cfg):
    c = N.StackConfig()
    for k, t in N.StackConfig._fields_:
        setattr(c, k, float(cfg[k]) if t is C.c_double else int(cfg[k]))
    layers = (N.LayerConfig * len(cfg["layers"]))()
    for dst, src in zip(layers, cfg["layers"]):
        for k, t in N.LayerConfig._fields_:  # what a layer does not name stays 0
            if k == "decay":
                if "decay" in src:
                    dst.decay = (C.c_double * len(src[k]))(*src[k])
            elif k in src:
                setattr(dst, k, float(src[k]) if t is C.c_double else int(src[k]))
    return c, layers


class Model:
    def __init__(self, ctx, cfg):
        self.ctx, self.cfg = ctx, dict(cfg)
        self.h = C.c_void_p()
        if cfg["arch"] == STACK:
            c, layers = make_stack_config(cfg)
            N.check(N.lib().strictb200_stack_create(ctx.h, C.byref(c), layers, C.byref(self.h)))
            return
        c = make_config(cfg)
        N.check(N.lib().strictb200_model_create(ctx.h, C.byref(c), C.byref(self.h)))

    def init_random(self, seed):
        N.check(N.lib().strictb200_model_init_random(self.h, seed))
        return self

    def set_tensor(self, name, host):
        host = np.ascontiguousarray(host)
        N.check(N.lib().strictb200_model_set_tensor(self.h, name.encode(), N.ptr(host), host.nbytes))

    def get_tensor(self, name, dtype, count):
        out = np.empty(count, dtype)
        N.check(N.lib().strictb200_model_get_tensor(self.h, name.encode(), N.ptr(out), out.nbytes))
        return out

    def weight_bytes(self):
        n = C.c_uint64()
        N.check(N.lib().strictb200_model_weight_bytes(self.h, C.byref(n)))
        return n.value

    def set_graph(self, enabled):
        N.check(N.lib().strictb200_model_set_graph(self.h, 1 if enabled else 0))

    def new_cache(self, batch, maxlen):
        return KvCache(self, batch, maxlen)

    def dispose(self):
        if self.h:
            N.lib().strictb200_model_destroy(self.h)
            self.h = C.c_void_p()

    Dispose = dispose


class KvCache:
    def __init__(self, model, batch, maxlen):
        self.model, self.B = model, batch
        self.h = C.c_void_p()
        N.check(N.lib().strictb200_kv_create(model.h, batch, maxlen, C.byref(self.h)))

    def reset(self):
        N.check(N.lib().strictb200_kv_reset(self.h))

    def lens(self):
        out = np.empty(self.B, np.int32)
        N.check(N.lib().strictb200_kv_lens(self.h, N.ptr(out)))
        return out

    def fill_synthetic(self, seed, length):
        N.check(N.lib().strictb200_kv_fill_synthetic(self.h, seed, length))

    def prefill(self, tokens, lens=None, want_logits=False):
        """tokens [B,S] int32; returns (next_ids[B], logits[B,V] or None)."""
        tokens = np.ascontiguousarray(tokens, dtype=np.int32)
        B, S = tokens.shape
        lens = np.full(B, S, np.int32) if lens is None else np.ascontiguousarray(lens, dtype=np.int32)
        nxt = np.empty(B, np.int32)
        logits = np.empty((B, self.model.cfg["vocab"]), np.float32) if want_logits else None
        N.check(N.lib().strictb200_prefill(self.model.h, self.h, N.ptr(tokens), N.ptr(lens), B, S, N.ptr(nxt), N.ptr(logits)))
        return nxt, logits

    def prefill_rows(self, tokens, want, lens=None):
        """tokens [B,S] int32 and, per sequence, the places among its new tokens whose logits are asked for;
        returns (next_ids[B], logits[places, V]), the sequences' places one after the other."""
        tokens = np.ascontiguousarray(tokens, dtype=np.int32)
        B, S = tokens.shape
        lens = np.full(B, S, np.int32) if lens is None else np.ascontiguousarray(lens, dtype=np.int32)
        n_want = np.array([len(w) for w in want], np.int32)
        places = np.array([p for w in want for p in w], np.int32)
        nxt = np.empty(B, np.int32)
        logits = np.empty((len(places), self.model.cfg["vocab"]), np.float32)
        N.check(N.lib().strictb200_prefill_rows(self.model.h, self.h, N.ptr(tokens), N.ptr(lens), B, S, N.ptr(places), N.ptr(n_want), N.ptr(nxt), N.ptr(logits)))
        return nxt, logits

    def decode_step(self, ids, want_logits=False, out=None):
        ids = np.ascontiguousarray(ids, dtype=np.int32)
        nxt = np.empty(self.B, np.int32) if out is None else out
        logits = np.empty((self.B, self.model.cfg["vocab"]), np.float32) if want_logits else None
        N.check(N.lib().strictb200_decode_step(self.model.h, self.h, N.ptr(ids), N.ptr(nxt), N.ptr(logits)))
        return nxt, logits

    def generate(self, ids, n_steps):
        ids = np.ascontiguousarray(ids, dtype=np.int32)
        out = np.empty((n_steps, self.B), np.int32)
        N.check(N.lib().strictb200_generate(self.model.h, self.h, N.ptr(ids), n_steps, N.ptr(out)))
        return out

    def decode_steps_device(self, n_steps):
        """n greedy steps with ids resident on the device (no host copies, asynchronous)."""
        N.check(N.lib().strictb200_decode_steps_device(self.model.h, self.h, None, n_steps))

    KERNEL_CLASSES = ("embed", "gemm_qkv", "rope_kvappend", "attn_decode", "gemm_o", "rownorm", "gemm_gate_up", "swiglu",
                      "gemm_down", "head", "allreduce", "attn_merge", "gates", "recurrence")

    def profile_decode(self, n_steps):
        """Per-kernel-class device time of n plain-launch decode steps: {class: (total_ms, calls)}."""
        ms = np.zeros(len(self.KERNEL_CLASSES), np.float32)
        calls = np.zeros(len(self.KERNEL_CLASSES), np.uint64)
        N.check(N.lib().strictb200_profile_decode(self.model.h, self.h, n_steps, N.ptr(ms), N.ptr(calls), len(ms)))
        return {k: (float(ms[i]), int(calls[i])) for i, k in enumerate(self.KERNEL_CLASSES)}

    def decode_bytes(self):
        n = C.c_uint64()
        N.check(N.lib().strictb200_decode_bytes(self.model.h, self.h, C.byref(n)))
        return n.value

    def dispose(self):
        if self.h:
            N.lib().strictb200_kv_destroy(self.h)
            self.h = C.c_void_p()

    Dispose = dispose
