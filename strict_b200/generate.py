"""Greedy generation from a model folder.

    python -m strict_b200.generate --model DIR --prompt 5,17,3 [--prompt 8,1] --new 32 [--dtype float32]

Every --prompt is one sequence of token ids; the prompts form one batch. Prints one line of new ids
per prompt.
"""
import argparse
import sys

import numpy as np


def greedy(model, prompts, new_tokens):
    """prompts: lists of ids of any lengths. Returns [len(prompts)][new_tokens] greedy ids."""
    lens = np.array([len(p) for p in prompts], np.int32)
    tokens = np.zeros((len(prompts), int(lens.max())), np.int32)
    for row, p in zip(tokens, prompts):
        row[:len(p)] = p
    kv = model.new_cache(len(prompts), int(lens.max()) + new_tokens)
    try:
        first, _ = kv.prefill(tokens, lens)
        if new_tokens == 1:
            return first[:, None]
        return np.concatenate([first[None], kv.generate(first, new_tokens - 1)]).T
    finally:
        kv.dispose()


def main(argv=None):
    ap = argparse.ArgumentParser(description="Greedy generation from a model folder.")
    ap.add_argument("--model", required=True)
    ap.add_argument("--prompt", action="append", required=True, help="comma-separated token ids; may be given several times")
    ap.add_argument("--new", type=int, default=16, help="tokens to generate per prompt")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    args = ap.parse_args(argv)
    from . import checkpoint, model as M
    from .kernel import Context
    prompts = [[int(t) for t in p.split(",")] for p in args.prompt]
    ctx = Context(0)
    model = checkpoint.load(ctx, args.model, max_pos=max(map(len, prompts)) + args.new, dtype=M.FP32 if args.dtype == "float32" else M.BF16)
    for row in greedy(model, prompts, args.new):
        print(",".join(str(int(t)) for t in row))
    model.dispose()
    ctx.dispose()
    return 0


if __name__ == "__main__":
    sys.exit(main())
