"""Replays a recorded trace of requests through a model folder and writes the logits asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps

Every line of standard input is one step, a JSON object

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["a"]}

A step feeds the next tokens of each entry's request to the request's cache: a single token after
the first goes through the decode step (the recorded CUDA graph that generation replays), anything
else through the prefill, which continues from what the cache holds. The logits at the wanted
places go to <out>/<step>.f32 (little-endian fp32, [wanted, vocab], in the order of the entries);
then "done <step>" is printed. Requests named in "end" give their cache back; it is reset and used
again.
"""
import argparse
import json
import os
import sys

import numpy as np


class Replay:
    def __init__(self, model, max_tokens):
        self.model, self.max_tokens = model, max_tokens
        self.live, self.free = {}, []  # request -> [cache, tokens it holds]; caches to use again

    def feed(self, name, tokens, want):
        """Logits [len(want), vocab] after the request's next tokens."""
        if name not in self.live:
            self.live[name] = [self.free.pop() if self.free else self.model.new_cache(1, self.max_tokens), 0]
        kv, held = self.live[name]
        self.live[name][1] += len(tokens)
        if len(tokens) == 1 and held > 0:
            _, logits = kv.decode_step(tokens, want_logits=bool(want))
            return np.repeat(logits, len(want), axis=0) if want else np.empty((0, self.model.cfg["vocab"]), np.float32)
        return kv.prefill_rows([tokens], [want])[1]

    def end(self, name):
        if name in self.live:
            kv, _ = self.live.pop(name)
            kv.reset()
            self.free.append(kv)

    def step(self, step):
        rows = [self.feed(e["id"], e["tokens"], e.get("want", [])) for e in step.get("entries", []) if e["tokens"]]
        for name in step.get("end", []):
            self.end(name)
        return np.concatenate(rows) if rows else np.empty((0, self.model.cfg["vocab"]), np.float32)


def main(argv=None):
    ap = argparse.ArgumentParser(description="Replay a trace of requests through a model folder and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the <step>.f32 files")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens that a request may hold")
    args = ap.parse_args(argv)
    from . import build
    build.build()  # does nothing when the library is up to date
    from . import checkpoint, model as M
    from .kernel import Context
    ctx = Context(0)
    model = checkpoint.load(ctx, args.model, max_pos=args.max_tokens, dtype=M.FP32 if args.dtype == "float32" else M.BF16)
    replay = Replay(model, args.max_tokens)
    for line in iter(sys.stdin.readline, ""):
        if not line.strip():
            continue
        step = json.loads(line)
        logits = replay.step(step)
        if len(logits):
            path = os.path.join(args.out, f"{step['step']}.f32")
            logits.astype("<f4").tofile(path)
        print(f"done {step['step']}", flush=True)
    for kv in [kv for kv, _ in replay.live.values()] + replay.free:
        kv.dispose()
    model.dispose()
    ctx.dispose()
    return 0
