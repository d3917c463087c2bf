"""Prefill and decode throughput of the Kipatar and Morarax designs at sizes that resemble a real model's layers (random
weights), beside the framework's closest existing model (Qwen3: grouped-query attention, sequential SwiGLU
layers, E4M3 weights) at equal width, depth, heads, feed-forward and vocabulary.

    python bench.py --design kipatar|morarax [--steps K] [--warmup W] [--sizes 8b,0.6b] [--layers N]

Prints one JSON line. A design whose layers have different mixers is also run with each mixer in every layer of a shorter
model (`mixers`): there the numbers of a kernel class belong to one mixer. Times are CUDA events on the library's stream (prefill: the public prefill call,
host ids in, greedy ids out; decode: graph-replayed steps with ids resident on the device). A step streams
more than L2 holds in every configuration but the few-layer ones of --layers. `kernels` are plain launches
of the decode step, one pair of events per call, with the bytes a call must move and their share of the
copy bandwidth, and beside it the same inside the replayed step (`exposed_us`, `hbm_frac_in_step`: how
far a launch moved the end of the chain, from per-block time stamps); `flops_frac` is a prefill's useful matrix work over the measured bf16 throughput.
"""
import json
import os

import numpy as np

from . import clocks, native as N, timeline
from .kernel import Context, DeviceVariable
from .model import (CONFIGS, MIXER_ATTENTION, MIXER_GATED, MIXER_LATENT, MLP_RELU_GLU, STACK, Model, attention_layer, gated_layer, latent_layer,
                    retention_layer, stack_config)

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))

# name -> (Qwen3 configuration, latent rank, rotated dims, window, [(batch, prompt)] for decode, for prefill)
SIZES = {
    "8b": ("qwen3-8b", 512, 64, 2048, [(32, 2048), (1, 2048)], [(8, 2048), (1, 2048), (1, 8192)]),
    "0.6b": ("qwen3-0.6b", 256, 64, 1024, [(32, 2048), (1, 2048)], [(8, 2048), (1, 2048)]),
}


def kipatar_like(qwen, rank, rot, window, max_pos):
    """The design at the sizes of a Qwen3 configuration: as many heads, heads as wide, the same feed-forward width. Every
    fourth layer reads the latents of the one before it."""
    layers = [latent_layer(heads=qwen["n_q_heads"], dim=qwen["head_dim"], rot_dim=rot, vdim=qwen["head_dim"], kv_rank=rank,
                           scale=(qwen["head_dim"] + rot) ** -0.5, rot_base=1e6, window=window, kv_from=i - 1 if i % 4 == 3 else -1, d_ff=qwen["d_ff"])
              for i in range(qwen["n_layers"])]
    return stack_config(layers, d_model=qwen["d_model"], vocab=qwen["vocab"], max_pos=max_pos, norm_groups=8, eps=1e-6)


def morarax_like(qwen, gate_blocks, max_pos, mixers):
    """The design at the sizes of a Qwen3 configuration: as many heads, heads as wide, the same feed-forward width, the gated
    recurrence as wide as the model. `mixers` are repeated over the layers."""
    H, D, d, ff = qwen["n_q_heads"], qwen["head_dim"], qwen["d_model"], qwen["d_ff"]
    make = {"attention": lambda: attention_layer(H, qwen["n_kv_heads"], D, D, D ** -0.5, rot_dim=D, rot_base=1e6, qk_norm=True, sink=True, gate=True, d_ff=ff,
                                                 rot_scaling=dict(factor=4.0, original=4096, fast=32.0, slow=1.0)),
            "gated": lambda: gated_layer(d, gate_blocks, 4, d_ff=ff),
            "retention": lambda: retention_layer(H, D, D, [1.0 - 2.0 ** (-5 - 7 * h / max(H - 1, 1)) for h in range(H)], rot_dim=D, rot_base=1e4, d_ff=ff)}
    layers = [make[mixers[i % len(mixers)]]() for i in range(qwen["n_layers"])]
    return stack_config(layers, d_model=d, vocab=qwen["vocab"], max_pos=max_pos, norm_groups=1, eps=1e-6, shared_norm=True, layer_scale=True, residual_mult=0.5)


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(path):
        p = json.load(open(path))
        return float(p["hbm_gbs"]), float(p["bf16_tflops"]), float(p.get("bf16_tflops_sustained", p["bf16_tflops"])), "measured"
    return 6650.0, 1590.0, 1400.0, "fallback"


def seen(n, window):
    """Sum over the positions 0..n-1 of the keys each sees."""
    w = window or n
    return sum(min(i + 1, w) for i in range(n)) if n < w else w * (w + 1) // 2 + (n - w) * w


def layer_parts(y, d):
    """Of one layer: rows of the input product, columns of the output product, other weights (elements), cache elements read per
    key, state floats per sequence."""
    ff = (2 if y["mlp"] == MLP_RELU_GLU else 1) * y["d_ff"]
    if y["mixer"] == MIXER_LATENT:
        H, q, own = y["heads"], y["dim"] + y["rot_dim"], y["kv_from"] < 0
        n_in = H * q + (y["kv_rank"] + y["rot_dim"] if own else 0)
        return n_in + ff, H * y["vdim"] + y["d_ff"], H * (y["dim"] + y["vdim"]) * y["kv_rank"], y["kv_rank"] + y["rot_dim"], 0
    if y["mixer"] == MIXER_GATED:
        w = y["width"]
        return 2 * w + ff, w + y["d_ff"], 2 * w * (w // y["blocks"]), 0, w * y["conv"]
    H, q, v = y["heads"], y["dim"], y["vdim"]
    if y["mixer"] == MIXER_ATTENTION:
        G = y["kv_heads"]
        return H * (q + 1) + G * (q + v) + ff, H * v + y["d_ff"], 0, G * (q + v), 0
    return 2 * H * (q + v) + ff, H * v + y["d_ff"], 0, 0, H * q * v


def prefill_flops(cfg, B, S):
    """Useful matrix work of a prompt: linear layers (the head on the last row only) and attention over the keys each position sees."""
    d, T, f = cfg["d_model"], B * S, 0
    if cfg["arch"] == STACK:
        for y in cfg["layers"]:
            n_in, n_out, other, _, state = layer_parts(y, d)
            f += 2 * T * (d * (n_in + n_out) + other)
            if y["mixer"] == MIXER_LATENT:
                f += 2 * B * seen(S, y["window"]) * y["heads"] * (y["dim"] + y["rot_dim"] + y["vdim"])
            elif y["mixer"] == MIXER_ATTENTION:
                f += 2 * B * seen(S, 0) * y["heads"] * (y["dim"] + y["vdim"])
            elif y["mixer"] != MIXER_GATED:
                f += 4 * T * state  # a state's update and its product with the query
        return f
    D, H, Hkv = cfg["head_dim"], cfg["n_q_heads"], cfg["n_kv_heads"]
    return cfg["n_layers"] * (2 * T * d * ((2 * H + 2 * Hkv) * D + 3 * cfg["d_ff"]) + 4 * B * seen(S, 0) * H * D)


def call_bytes(cfg, B, length):
    """Bytes a call of each kernel class of the decode step must move (weights or cache once), averaged over the layers."""
    d = cfg["d_model"]
    if cfg["arch"] == STACK:
        L = cfg["layers"]
        mean = lambda f: sum(f(y) for y in L) / len(L)  # noqa: E731
        parts = lambda i: mean(lambda y: layer_parts(y, d)[i])  # noqa: E731
        out = {"gemm_qkv": 2 * d * parts(0), "gemm_o": 2 * d * parts(1), "head": 2 * cfg["vocab"] * d}
        kinds = {y["mixer"] for y in L}
        if kinds == {MIXER_LATENT}:
            out.update({"rope_kvappend": 2 * mean(lambda y: y["heads"] * y["dim"] * y["kv_rank"]),
                        "attn_decode": 2 * B * mean(lambda y: min(length, y["window"] or length) * (y["kv_rank"] + y["rot_dim"])),
                        "attn_merge": 2 * mean(lambda y: y["heads"] * y["vdim"] * y["kv_rank"])})
        elif len(kinds) == 1:
            out.update({"attn_decode": 2 * B * length * parts(3), "gates": 2 * parts(2), "recurrence": 8 * B * parts(4)})
        return {k: v for k, v in out.items() if v}
    D, H, Hkv, I = cfg["head_dim"], cfg["n_q_heads"], cfg["n_kv_heads"], cfg["d_ff"]
    return {"gemm_qkv": (H + 2 * Hkv) * D * d, "gemm_o": H * D * d, "gemm_gate_up": 2 * I * d, "gemm_down": d * I, "head": cfg["vocab"] * d,
            "attn_decode": B * length * Hkv * D * 4}


TRACE_CLASS = {"rope": "rope_kvappend", "attn_combine": "attn_merge"}


def gemm_names(cfg):
    """(N, K) of the decode step's GEMM launches -> kernel class, to label them in a trace."""
    d = cfg["d_model"]
    if cfg["arch"] != STACK:
        D, H, Hkv, I = cfg["head_dim"], cfg["n_q_heads"], cfg["n_kv_heads"], cfg["d_ff"]
        return {((H + 2 * Hkv) * D, d): "gemm_qkv", (d, H * D): "gemm_o", (2 * I, d): "gemm_gate_up", (d, I): "gemm_down", (cfg["vocab"], d): "head"}
    out = {(cfg["vocab"], d): "head"}
    for y in cfg["layers"]:
        n_in, n_out, _, _, _ = layer_parts(y, d)
        ff = (2 if y["mlp"] == MLP_RELU_GLU else 1) * y["d_ff"]
        out[(-(-(n_in - ff) // 256) * 256 + ff, d)] = "gemm_qkv"
        out[(d, n_out)] = "gemm_o"
        if y["mixer"] == MIXER_GATED:
            out[(2 * y["width"], y["width"] // y["blocks"])] = "gates"
    return out


def ids(ctx, n, vocab, seed):
    v = DeviceVariable(ctx, n, np.int32)
    N.check(N.lib().strictb200_gen_tokens(ctx.h, seed, 1, n, vocab, v.p))
    out = v.to_host()
    v.free()
    return out


def run_model(ctx, cfg, decode, prefill, steps, warmup):
    hbm, burst, sustained, _ = peaks()
    model = Model(ctx, cfg).init_random(5)
    out = {"weights_gb": model.weight_bytes() / 1e9, "prefill": [], "decode": []}
    for B, S in prefill:
        toks = ids(ctx, B * S, cfg["vocab"], 6).reshape(B, S)
        kv = model.new_cache(B, S)
        for _ in range(3):
            kv.reset()
            kv.prefill(toks)
        times = []
        sampler = clocks.ClockSampler(0)
        sampler.start()
        for _ in range(max(3, min(steps, 5))):
            kv.reset()
            ctx.synchronize()
            ctx.timer_begin()
            kv.prefill(toks)
            times.append(ctx.timer_end())
        ms, flops = float(np.median(times)), prefill_flops(cfg, B, S)
        out["prefill"].append({"batch": B, "prompt": S, "ms": ms, "tokens_per_s": B * S / ms * 1e3, "tflops": flops / ms / 1e9,
                               "flops_frac": flops / ms / 1e9 / sustained, "clocks": sampler.stop()})
        kv.dispose()
    for B, S in decode:
        kv = model.new_cache(B, S + 2 * (steps + warmup) + 16)
        kv.fill_synthetic(7, S)
        kv.decode_step(ids(ctx, B, cfg["vocab"], 8))
        kv.decode_steps_device(max(3, warmup))
        ctx.synchronize()
        sampler = clocks.ClockSampler(0)
        sampler.start()
        nbytes = kv.decode_bytes()
        ctx.timer_begin()
        kv.decode_steps_device(steps)
        ms = ctx.timer_end() / steps
        clk = sampler.stop()
        kernels, per_call = {}, call_bytes(cfg, B, int(kv.lens().mean()))
        for k, (tot, calls) in kv.profile_decode(3).items():
            if calls:
                us = tot / calls * 1e3
                kernels[k] = {"us": us, "calls_per_step": calls / 3}
                if k in per_call:
                    calls_of_bytes = calls / 3 if k != "head" else 1  # the head's product and its pick are two calls
                    kernels[k]["hbm_frac"] = per_call[k] / (tot * 1e3 / (3 * calls_of_bytes) * 1e-6) / 1e9 / hbm
        # the same classes inside the replayed step, from the kernels' own time stamps: how far each launch moved the end of the chain
        with ctx.trace(1 << 20) as tr:
            kv.decode_steps_device(1)
        for k, (ns, calls) in timeline.per_kernel(timeline.launches(tr.records, gemm_names(cfg))).items():
            k = TRACE_CLASS.get(k, k)
            if k in kernels:
                e = kernels[k]
                e["exposed_us"] = e.get("exposed_us", 0.0) + ns / 1e3 / e["calls_per_step"]
        for k, e in kernels.items():
            if k in per_call and e.get("exposed_us") and k != "head":
                e["hbm_frac_in_step"] = per_call[k] / (e["exposed_us"] * 1e-6) / 1e9 / hbm
        out["decode"].append({"batch": B, "context": S, "ms": ms, "tokens_per_s": B / ms * 1e3, "step_gb": nbytes / 1e9,
                              "hbm_frac": nbytes / (ms * 1e-3) / 1e9 / hbm, "kernels": kernels, "clocks": clk})
        kv.dispose()
    ctx.device_status()
    model.dispose()
    return out


# name -> (Qwen3 configuration, gate blocks); batches and prompts as above
MORARAX = {"8b": ("qwen3-8b", 16), "0.6b": ("qwen3-0.6b", 8)}
ORDER = ("gated", "retention", "retention", "attention")


def run(design, sizes, steps, warmup, layers=0):
    ctx = Context(0)
    hbm, burst, sustained, kind = peaks()
    result = {"design": design, "data": "synthetic (random weights)", "peaks": {"hbm_gbs": hbm, "bf16_tflops": burst, "bf16_tflops_sustained": sustained, "kind": kind},
              "steps": steps, "warmup": warmup, "sizes": {}}
    for name in sizes:
        base, rank, rot, window, decode, prefill = SIZES[name]
        qwen = dict(CONFIGS[base], max_pos=16384)
        if layers:
            qwen["n_layers"] = layers
        config = {"width": qwen["d_model"], "layers": qwen["n_layers"], "heads": qwen["n_q_heads"], "dim": qwen["head_dim"], "ff": qwen["d_ff"], "vocab": qwen["vocab"]}
        out = result["sizes"][name] = {"config": config}
        if design == "kipatar":
            config.update({"rot_dim": rot, "kv_rank": rank, "window": window, "norm_groups": 8, "kv_from": "every fourth layer"})
            out[design] = run_model(ctx, kipatar_like(qwen, rank, rot, window, 16384), decode, prefill, steps, warmup)
        else:
            blocks = MORARAX[name][1]
            config.update({"kv_heads": qwen["n_kv_heads"], "gate_blocks": blocks, "conv": 4, "order": ORDER})
            out[design] = run_model(ctx, morarax_like(qwen, blocks, 16384, ORDER), decode, prefill, steps, warmup)
            out["mixers"] = {m: run_model(ctx, morarax_like(dict(qwen, n_layers=min(8, qwen["n_layers"])), blocks, 16384, (m,)), decode, prefill, steps, warmup)
                             for m in dict.fromkeys(ORDER)}
        out["qwen3"] = run_model(ctx, qwen, decode, prefill, steps, warmup)
    ctx.dispose()
    print(json.dumps(result), flush=True)
