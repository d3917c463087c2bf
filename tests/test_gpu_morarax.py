"""Morarax on the GPU against the plain implementation (plain_morarax.py, float64): every mechanism alone, whole prompts, prompts
in portions, token-by-token decoding, unequal batches, caches and states used again, keys and memories that stand out, long
decoding, greedy generation, in bf16 and in fp32.

The error of a row of logits is the root mean square of its difference (mean taken off) over that of the reference row. fp32
rounding alone gives about 1e-6, bf16 about 5e-3 for these models."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import morarax_models as MM
import plain_morarax as P
import strict_b200 as sb
from strict_b200 import checkpoint, generate

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
LIMIT = {sb.FP32: 3e-5, sb.BF16: 3e-2}
dtypes = pytest.mark.parametrize("dtype", [sb.FP32, sb.BF16], ids=["fp32", "bf16"])
_weights, _plain = {}, {}


def weights_of(name):
    if name not in _weights:
        _weights[name] = MM.weights(MM.CONFIGS[name], 11)
    return _weights[name]


def tokens_of(name, n, seed=5):
    return np.random.default_rng(seed).integers(0, MM.CONFIGS[name]["vocab"], n).astype(np.int32)


def plain(name, tokens):
    key = (name, tuple(int(t) for t in tokens))
    if key not in _plain:
        _plain[key] = P.forward(MM.CONFIGS[name], weights_of(name), tokens)
    return _plain[key]


def make(ctx, cfg, w, dtype, max_pos=2048):
    m = sb.Model(ctx, checkpoint.ARCHITECTURES["Morarax"](cfg, max_pos, dtype))
    for k, v in w.items():
        m.set_tensor(k, MM.bf16_bits(v))
    return m


@pytest.fixture(scope="module")
def models(ctx):
    made = {}

    def get(name, dtype):
        if (name, dtype) not in made:
            made[name, dtype] = make(ctx, MM.CONFIGS[name], weights_of(name), dtype)
        return made[name, dtype]

    yield get
    for m in made.values():
        m.dispose()


def row_errors(got, want):
    d = np.asarray(got, np.float64) - want
    d -= d.mean(-1, keepdims=True)
    c = want - want.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1) / (c * c).mean(-1))


def check(got, want, dtype, what=""):
    assert got.shape == want.shape
    e = row_errors(got, want)
    assert e.max() <= LIMIT[dtype], (what, int(e.argmax()), float(e.max()))


def portions(kv, tokens, sizes):
    """Feeds the tokens in portions (single tokens through the decode step), returns all logits."""
    rows, at = [], 0
    for n in sizes:
        part = tokens[at:at + n]
        if len(part) == 1 and at:
            rows.append(kv.decode_step(part, want_logits=True)[1])
        else:
            rows.append(kv.prefill_rows([part], [range(len(part))])[1])
        at += n
    assert at == len(tokens)
    return np.concatenate(rows)


# ------------------------------------------------------------------ mechanisms alone
def _alone(entry, width=64, **kw):
    return MM.config([entry], width, 50, **kw)


ONE = {  # one part of the layer at a time, with the sizes that matter to it
    "heads that share keys": _alone(MM.attention(6, 2, 16, 24, MM.rot(300.0, 8), 0)),
    "sixteen heads on one key": _alone(MM.attention(16, 1, 64, 64, MM.rot(300.0, 64), 0)),
    "more heads on a key than a tile has rows": _alone(MM.attention(20, 1, 32, 32, MM.rot(300.0, 32), 0)),
    "hardly any rotation": _alone(MM.attention(2, 2, 48, 16, MM.rot(9000.0, 2), 0)),
    "stretched rotation": _alone(MM.attention(2, 1, 64, 32, MM.rot(10000.0, 64, 16.0, original=32, fast=4.0, slow=0.25), 0)),
    "stretched rotation of a part": _alone(MM.attention(2, 1, 32, 32, MM.rot(200.0, 12, 3.0), 0)),
    "a stretch without a ramp": _alone(MM.attention(2, 1, 32, 32, MM.rot(200.0, 32, 3.0, fast=1.0, slow=1.0), 0)),
    "a scale": _alone(MM.attention(2, 1, 16, 16, MM.rot(200.0, 16), 0, scale=1.7)),
    "a large epsilon": _alone(MM.attention(2, 1, 16, 16, MM.rot(200.0, 16), 0), eps=0.3),
    "wide values": _alone(MM.attention(3, 3, 24, 112, MM.rot(200.0, 24), 0)),
    "wide keys": _alone(MM.attention(3, 3, 120, 20, MM.rot(200.0, 60), 0)),
    "a convolution of one tap": _alone(MM.rglru(48, 2, 1, 0)),
    "a long convolution": _alone(MM.rglru(40, 2, 9, 0)),
    "one gate block": _alone(MM.rglru(64, 1, 4, 0)),
    "gate blocks of two channels": _alone(MM.rglru(32, 16, 3, 0)),
    "gate blocks that fill a tile": _alone(MM.rglru(512, 4, 4, 0)),
    "retention of one head": _alone(MM.retention(1, 32, 16, MM.rot(100.0, 32), 0)),
    "retention under many decays": _alone(MM.retention(6, 16, 48, MM.rot(100.0, 8), 0, decay=[0.0, 0.25, 0.9, 0.99, 0.9995, 1.0])),
    "retention, wide values": _alone(MM.retention(2, 20, 128, MM.rot(100.0, 20), 0)),
    "a feed-forward": _alone(MM.rglru(8, 1, 1, 136)),
    "a feed-forward of odd width": _alone(MM.rglru(8, 1, 1, 131)),
    "no scales": _alone(MM.retention(2, 16, 16, MM.rot(100.0, 16), 24), residual_mult=1.0, logit_scale=1.0),
}


@dtypes
@pytest.mark.parametrize("what", list(ONE))
def test_one_mechanism(ctx, what, dtype):
    cfg = ONE[what]
    w = MM.weights(cfg, 2, 3.0)
    t = np.random.default_rng(8).integers(0, cfg["vocab"], 150).astype(np.int32)
    want = P.forward(cfg, w, t)
    m = make(ctx, cfg, w, dtype, 160)
    kv = m.new_cache(1, 160)
    for sizes in ([150], [70] + [1] * 30 + [50], [1] * 20 + [130], [3, 2, 140, 5]):
        kv.reset()
        check(portions(kv, t, sizes), want, dtype, sizes[:3])
    kv.dispose(), m.dispose()


# ------------------------------------------------------------------ prompts, decoding, portions
@dtypes
@pytest.mark.parametrize("name,n", [("mixed", 330), ("odd", 150), ("tiles", 400), ("wide", 140), ("one", 200)])
def test_whole_prompts(models, name, n, dtype):
    t = tokens_of(name, n)
    kv = models(name, dtype).new_cache(1, n)
    nxt, logits = kv.prefill_rows([t], [range(n)])
    check(logits, plain(name, t), dtype)
    assert nxt[0] == logits[-1].argmax()
    kv.dispose()


@dtypes
@pytest.mark.parametrize("name,n,first", [("mixed", 330, 1), ("odd", 150, 1), ("tiles", 300, 190), ("wide", 70, 20), ("one", 200, 2)])
def test_decoding_token_by_token(models, name, n, first, dtype):
    t = tokens_of(name, n)
    kv = models(name, dtype).new_cache(1, n)
    check(portions(kv, t, [first] + [1] * (n - first)), plain(name, t), dtype)
    assert kv.lens().tolist() == [n]
    kv.dispose()


SIZES = {"pairs": [2] * 150, "threes": [3] * 100, "mixed": [5, 1, 2, 1, 1, 31, 2, 64, 2, 1, 150, 40], "chunk edges": [127, 2, 126, 1, 2, 42],
         "chunk": [128, 128, 44], "one more than a chunk": [129, 129, 42], "two and rest": [2, 298]}


@dtypes
@pytest.mark.parametrize("sizes", list(SIZES))
@pytest.mark.parametrize("name", ["mixed", "odd", "tiles"])
def test_portions(models, name, sizes, dtype):
    t = tokens_of(name, 300)
    kv = models(name, dtype).new_cache(1, 300)
    check(portions(kv, t, SIZES[sizes]), plain(name, t), dtype)
    kv.dispose()


@dtypes
def test_batches_of_unequal_requests(ctx, models, dtype):
    name, lens, n = "mixed", [130, 1, 64, 129, 7, 200], 12
    m = models(name, dtype)
    prompts = [tokens_of(name, k, 20 + k) for k in lens]
    more = np.random.default_rng(3).integers(0, MM.CONFIGS[name]["vocab"], (n, len(lens))).astype(np.int32)
    want = [plain(name, np.concatenate([p, more[:, b]])) for b, p in enumerate(prompts)]
    tok = np.zeros((len(lens), max(lens)), np.int32)
    for row, p in zip(tok, prompts):
        row[:len(p)] = p
    tail = [tokens_of(name, k, 70 + k) for k in (3, 2, 40, 1, 9, 2)]
    pad = np.zeros((len(lens), 40), np.int32)
    for row, p in zip(pad, tail):
        row[:len(p)] = p
    try:
        for chunk in (16384, 140):  # one prefill chunk, and several of one or more sequences
            ctx.set_option("prefill_chunk", chunk)
            kv = m.new_cache(len(lens), 260)
            places = [sorted({0, k // 2, k - 1}) for k in lens]
            _, logits = kv.prefill_rows(tok, places, lens)
            check(logits, np.concatenate([w[p] for w, p in zip(want, places)]), dtype, "prompt")
            for s in range(n):
                _, logits = kv.decode_step(more[s], want_logits=True)
                check(logits, np.stack([w[k + s] for w, k in zip(want, lens)]), dtype, s)
            # a second portion for all of them, again of unequal lengths
            _, logits = kv.prefill(pad, [len(p) for p in tail], want_logits=True)
            check(logits, np.stack([plain(name, np.concatenate([p, more[:, b], q]))[-1] for b, (p, q) in enumerate(zip(prompts, tail))]), dtype, "second portion")
            kv.dispose()
    finally:
        ctx.set_option("prefill_chunk", 16384)


@pytest.mark.parametrize("B", [33, 130, 260])
@pytest.mark.parametrize("name", ["odd", "tiles"])
def test_many_sequences(models, B, name):
    """Decode batches of more than one token group, more than 128 and more than 256 rows, over different lengths."""
    lens = np.array([1 + (7 * b) % 23 for b in range(B)], np.int32)
    tok = np.stack([tokens_of(name, 24, b % 9) for b in range(B)])
    kv = models(name, sb.BF16).new_cache(B, 32)
    kv.prefill(tok, lens)
    nxt, logits = kv.decode_step(tok[np.arange(B), lens], want_logits=True)
    check(logits, np.stack([plain(name, tok[b])[lens[b]] for b in range(B)]), sb.BF16)
    assert np.array_equal(nxt, logits.argmax(1))
    kv.dispose()


@dtypes
@pytest.mark.parametrize("name", ["mixed", "tiles"])
def test_a_cache_used_again(models, name, dtype):
    m = models(name, dtype)
    t, other = tokens_of(name, 90), tokens_of(name, 200, 99)
    sizes = [50, 2, 1, 30] + [1] * 7
    fresh = m.new_cache(1, 256)
    want = portions(fresh, t, sizes)
    used = m.new_cache(1, 256)
    portions(used, other, [150] + [1] * 50)
    used.reset()
    got = portions(used, t, sizes)
    assert np.array_equal(got, want)
    check(got, plain(name, t), dtype)
    # the place in a batch does not matter either
    three = m.new_cache(3, 256)
    three.prefill(np.stack([other[:60], t[:60], other[60:120]]))
    logits = [three.decode_step([0, t[i], 1], want_logits=True)[1][1] for i in range(60, 90)]
    check(np.stack(logits), plain(name, t)[60:], dtype)
    for kv in (fresh, used, three):
        kv.dispose()


def test_two_caches_side_by_side(models):
    """Steps of two requests in turn, as a replayed trace makes them."""
    m = models("mixed", sb.BF16)
    a, b = tokens_of("mixed", 60, 1), tokens_of("mixed", 60, 2)
    ka, kb = m.new_cache(1, 64), m.new_cache(1, 64)
    got = {0: [], 1: []}
    for lo, n in ((0, 20), (20, 1), (21, 1), (22, 1), (23, 30), (53, 1), (54, 6)):
        for i, (kv, t) in enumerate(((ka, a), (kb, b))):
            part = t[lo:lo + n]
            got[i].append(kv.decode_step(part, want_logits=True)[1] if n == 1 else kv.prefill_rows([part], [range(n)])[1])
    for i, t in enumerate((a, b)):
        check(np.concatenate(got[i]), plain("mixed", t), sb.BF16, i)
    ka.dispose(), kb.dispose()


@pytest.mark.parametrize("lens", [[700], [1100, 300, 129, 5], [513, 512, 511, 1]])
def test_long_prompts_in_segments(ctx, lens):
    """Few heads and long prompts: retention cuts them into segments that run side by side; whole, continued, and decoded on."""
    cfg = MM.config([MM.retention(2, 64, 96, MM.rot(800.0, 64), 24, decay=[0.98, 0.9997]), MM.retention(3, 128, 40, MM.rot(800.0, 32), 0)], 96, 50)
    w = MM.weights(cfg, 12)
    rng = np.random.default_rng(6)
    seqs = [rng.integers(0, 50, n + 290).astype(np.int32) for n in lens]
    want = [P.forward(cfg, w, t) for t in seqs]
    m = make(ctx, cfg, w, sb.BF16)
    kv = m.new_cache(len(lens), max(lens) + 320)

    def feed(lo, n):
        tok = np.zeros((len(seqs), max(n)), np.int32)
        for row, t, a, k in zip(tok, seqs, lo, n):
            row[:k] = t[a:a + k]
        _, logits = kv.prefill_rows(tok, [range(k) for k in n], n)
        check(logits, np.concatenate([x[a:a + k] for x, a, k in zip(want, lo, n)]), sb.BF16, (lo, n))

    feed([0] * len(lens), lens)
    feed(lens, [280] * len(lens))
    for i in range(10):
        _, logits = kv.decode_step([t[n + 280 + i] for t, n in zip(seqs, lens)], want_logits=True)
        check(logits, np.stack([x[n + 280 + i] for x, n in zip(want, lens)]), sb.BF16, i)
    kv.dispose(), m.dispose()


# ------------------------------------------------------------------ keys and memories that stand out
def standing_out(seed):
    """One attention layer in which one token's key stands out for one query token, whatever the distance: little of a head is
    rotated, and the scale makes the pair's score large. Returns config, weights and the pair (query id, key id)."""
    cfg = MM.config([MM.attention(2, 1, 32, 32, MM.rot(1e5, 2), 0)], 96, 40, residual_mult=2.0)
    w = MM.weights(cfg, seed)
    h = P.rms(w["embed"].astype(np.float64), cfg["norm"]["eps"]) * w["l0.norm1"]
    q = P.rms((h @ w["l0.mix.q"].T).reshape(40, 2, 32), cfg["norm"]["eps"])
    k = P.rms((h @ w["l0.mix.k"].T).reshape(40, 32), cfg["norm"]["eps"])
    s = np.einsum("ahd,bd->ab", q[:, :1, 2:], k[:, 2:])
    a, b = np.unravel_index(s.argmax(), s.shape)
    cfg["layers"][0]["mixer"]["scale"] = float(18.0 / s.max())
    return cfg, w, int(a), int(b)


@dtypes
def test_a_far_key_weighs(ctx, dtype):
    cfg, w, ask, key = standing_out(21)
    filler = [t for t in range(40) if t not in (ask, key)]
    rng = np.random.default_rng(0)
    m = make(ctx, cfg, w, dtype, 1024)
    kv = m.new_cache(1, 1024)
    for at, distance in ((0, 1), (0, 63), (0, 64), (1, 127), (0, 128), (62, 2), (63, 1), (64, 200), (127, 1), (127, 2), (128, 129), (5, 600), (255, 300)):
        t = rng.choice(filler, at + distance + 3).astype(np.int32)
        row = at + distance
        t[at], t[row] = key, ask
        want = P.forward(cfg, w, t)
        gone = t.copy()
        gone[at] = filler[0]
        assert row_errors(P.forward(cfg, w, gone), want)[row] > 5 * LIMIT[dtype]  # without that key the row is another one
        for sizes in ([len(t)], [row] + [1] * 3, [max(1, row - 1), 2, 2] if row > 1 else [len(t)]):
            kv.reset()
            check(portions(kv, t, sizes)[row:row + 1], want[row:row + 1], dtype, (at, distance, sizes))
    kv.dispose(), m.dispose()


@dtypes
def test_the_sink_takes_its_share(ctx, dtype, monkeypatch):
    """Where all scores are low the sink takes most of the weight: first tokens, prompt and decode."""
    cfg = MM.config([MM.attention(4, 2, 32, 32, MM.rot(1e3, 32), 0, scale=0.02)], 96, 40, residual_mult=2.0)
    w = MM.weights(cfg, 4)
    t = np.random.default_rng(1).integers(0, 40, 12).astype(np.int32)
    want = P.forward(cfg, w, t)
    with monkeypatch.context() as p:
        def without(scores, mask):
            e = np.where(mask, np.exp(scores), 0.0)
            return e / e.sum(-1, keepdims=True)
        p.setattr(P, "softmax_with_sink", without)
        assert row_errors(P.forward(cfg, w, t), want)[:4].min() > 3 * LIMIT[sb.BF16]
    m = make(ctx, cfg, w, dtype, 64)
    kv = m.new_cache(1, 64)
    for sizes in ([12], [1] * 12, [2, 1, 9]):
        kv.reset()
        check(portions(kv, t, sizes), want, dtype, sizes)
    kv.dispose(), m.dispose()


MEMORIES = {  # layers that remember one early token for hundreds of positions
    "retention": (MM.config([MM.retention(2, 32, 32, MM.rot(1e6, 4), 0, decay=[0.9998, 1.0])], 96, 40, residual_mult=0.7), {}),
    "retention of full tiles": (MM.config([MM.retention(2, 128, 128, MM.rot(1e6, 8), 0, decay=[0.9998, 1.0])], 96, 40, residual_mult=0.7), {}),
    "gated recurrence": (MM.config([MM.rglru(96, 2, 3, 0)], 96, 40, residual_mult=2.0), {"forget": -6.0}),
}


@dtypes
@pytest.mark.parametrize("what", list(MEMORIES))
def test_an_early_token_is_remembered(ctx, what, dtype):
    """One loud token among quiet ones, at a chunk's edge or first: rows a hundred positions later still depend on it."""
    cfg, kw = MEMORIES[what]
    w = MM.weights(cfg, 9, **kw)
    loud = 7
    h = P.rms(w["embed"].astype(np.float64), cfg["norm"]["eps"]) * w["l0.norm1"]
    value = "l0.mix.v" if "l0.mix.v" in w else "l0.mix.x"
    # what enters the memory is large for one token only
    w[value] = MM.round_bf16(w[value] + np.outer(np.random.default_rng(77).standard_normal(len(w[value])), h[loud] / np.linalg.norm(h[loud])))
    rng = np.random.default_rng(3)
    quiet = [t for t in range(40) if t != loud]
    m = make(ctx, cfg, w, dtype, 512)
    kv = m.new_cache(1, 512)
    for at in (0, 1, 126, 127, 128, 255, 256):
        n = at + 200
        t = rng.choice(quiet, n).astype(np.int32)
        t[at] = loud
        want = P.forward(cfg, w, t)
        gone = t.copy()
        gone[at] = quiet[0]
        assert row_errors(P.forward(cfg, w, gone), want)[at + 100:].max() > 2.5 * LIMIT[dtype]
        for sizes in ([n], [at + 1, n - at - 1] if at else [n], [n - 40] + [1] * 40, [128] * (n // 128) + ([n % 128] if n % 128 else [])):
            kv.reset()
            check(portions(kv, t, sizes), want, dtype, (at, sizes[:3]))
    kv.dispose(), m.dispose()


@dtypes
def test_long_decoding(models, dtype):
    name, n = "odd", 700
    t = tokens_of(name, n, 44)
    kv = models(name, dtype).new_cache(1, n)
    check(portions(kv, t, [5] + [1] * (n - 5)), plain(name, t), dtype)
    kv.dispose()


@dtypes
def test_portions_agree_beyond_rounding(models, dtype):
    """The same rows however the prompt is cut, to a few times the rounding and not to the limit of the tests above."""
    t = tokens_of("tiles", 300)
    kv = models("tiles", dtype).new_cache(1, 300)
    whole = portions(kv, t, [300]).astype(np.float64)
    for sizes in ([2] * 150, [128, 44, 128], [299, 1]):
        kv.reset()
        e = row_errors(portions(kv, t, sizes), whole)
        assert e.max() <= (2e-6 if dtype == sb.FP32 else 1.2e-2), (sizes[:2], e.max())
    kv.dispose()


# ------------------------------------------------------------------ generation, folders, replay
@dtypes
def test_greedy_generation(models, dtype):
    name, new = "mixed", 24
    prompts = [tokens_of(name, k, 50 + k).tolist() for k in (9, 1, 70)]
    got = generate.greedy(models(name, dtype), prompts, new)
    for ids, p in zip(got, prompts):
        picks, margins = P.greedy(MM.CONFIGS[name], weights_of(name), p, new)
        for s in range(new):
            if ids[s] != picks[s]:
                assert margins[s] < (1e-3 if dtype == sb.FP32 else 0.1), (s, margins[s])  # a near tie: the paths part here
                break


def test_plain_launches_and_graph_agree(models):
    m = models("mixed", sb.BF16)
    t = tokens_of("mixed", 100)
    out = []
    for graph in (True, False):
        m.set_graph(graph)
        kv = m.new_cache(1, 100)
        out.append(portions(kv, t, [60] + [1] * 40))
        kv.dispose()
    m.set_graph(True)
    assert np.array_equal(out[0], out[1])


@dtypes
@pytest.mark.parametrize("name", ["odd", "tiles"])
def test_tensors_round_trip(models, name, dtype):
    m = models(name, dtype)
    for k, v in weights_of(name).items():
        assert np.array_equal(m.get_tensor(k, np.float32, v.size).reshape(v.shape), v), k
        assert np.array_equal(m.get_tensor(k, np.uint16, v.size).reshape(v.shape), MM.bf16_bits(v)), k
    for bad in ("l0.norm2", "l0.mix.dkv", "l0.mix", "l0.mlp.act"):
        with pytest.raises(ValueError):
            m.set_tensor(bad, np.zeros(4, np.float32))


def test_configurations_that_are_refused(ctx):
    good = checkpoint.ARCHITECTURES["Morarax"](MM.CONFIGS["mixed"], 64, sb.BF16)
    for layer, key, value in ((0, "kv_heads", 3), (0, "rot_dim", 42), (0, "rot_dim", 7), (0, "scale", 0.0), (0, "rot_slow", 0.0), (1, "blocks", 5), (1, "conv", 0),
                              (2, "decay", [0.5, 0.5, 1.5]), (2, "heads", 0)):
        bad = copy.deepcopy(good)
        bad["layers"][layer][key] = value
        with pytest.raises(ValueError):
            sb.Model(ctx, bad)
    for key in ("residual_mult", "logit_scale"):
        with pytest.raises(ValueError):
            sb.Model(ctx, dict(good, **{key: 0.0}))


def test_folder_and_replay(tmp_path):
    """bin/trace_run in a process of its own: portions, single tokens, wanted places, a second request after the first."""
    name = "odd"
    cfg, w = MM.CONFIGS[name], weights_of(name)
    MM.write_folder(tmp_path, cfg, w)
    a, b = tokens_of(name, 40, 1), tokens_of(name, 30, 2)
    plan = [("a", 0, 17, [0, 16]), ("a", 17, 2, [1]), ("a", 19, 1, [0]), ("a", 20, 1, []), ("a", 21, 19, [18, 3]), ("b", 0, 1, [0]), ("b", 1, 1, [0]), ("b", 2, 28, [27])]
    seqs = {"a": a, "b": b}
    for dtype, flag in ((sb.BF16, "bfloat16"), (sb.FP32, "float32")):
        out = tmp_path / flag
        out.mkdir()
        lines = [json.dumps({"step": i, "entries": [{"id": r, "tokens": seqs[r][lo:lo + n].tolist(), "want": want}],
                             "end": [r] if lo + n == len(seqs[r]) else []}) for i, (r, lo, n, want) in enumerate(plan)]
        p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", flag, "--out", str(out), "--max-tokens", "40"],
                           input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=600)
        assert p.returncode == 0, p.stderr[-2000:]
        for i, (r, lo, n, want) in enumerate(plan):
            path = out / f"{i}.f32"
            assert path.exists() == bool(want)
            if want:
                check(np.fromfile(path, "<f4").reshape(len(want), -1), plain(name, seqs[r])[[lo + k for k in want]], dtype, i)
    p = subprocess.run([sys.executable, "-m", "strict_b200.generate", "--model", str(tmp_path), "--prompt", "1,2,3", "--prompt", "4", "--new", "5", "--dtype", "float32"],
                       capture_output=True, text=True, timeout=600, cwd=ROOT)
    assert p.returncode == 0, p.stderr[-2000:]
    ids = [[int(x) for x in line.split(",")] for line in p.stdout.split()]
    assert [len(x) for x in ids] == [5, 5] and ids[0] == P.greedy(cfg, w, [1, 2, 3], 5)[0]


# ------------------------------------------------------------------ a latent mixer beside the others
@dtypes
def test_mixers_of_two_designs_in_one_stack(ctx, dtype):
    """Latent attention between a gated recurrence and retention, under the gated feed-forward and the scales per channel."""
    import plain_layered as PL
    d, vocab = 96, 60
    cfg = MM.config([MM.rglru(48, 2, 3, 40), MM.retention(2, 16, 24, MM.rot(300.0, 16), 32)], d, vocab)
    w = MM.weights(cfg, 31)
    rng = np.random.default_rng(32)
    latent = dict(heads=3, dim=16, rot_dim=8, vdim=24, kv_rank=32, scale=0.2, rot_base=500.0, window=20, d_ff=56)
    shapes = {"mix.q": (72, d), "mix.dkv": (40, d), "mix.uk": (48, 32), "mix.uv": (72, 32), "mix.o": (d, 72), "mlp.gate": (56, d), "mlp.up": (56, d), "mlp.down": (d, 56)}
    lw = {k: MM.round_bf16(rng.standard_normal(s) / np.sqrt(s[1])) for k, s in shapes.items()}
    for k, n in (("norm1", d), ("ls1", d), ("ls2", d), ("mix.dkv.norm", 32)):
        lw[k] = MM.round_bf16(1.0 + 0.3 * rng.standard_normal(n))
    base = checkpoint.ARCHITECTURES["Morarax"](cfg, 160, dtype)
    layers = [base["layers"][0], dict(sb.latent_layer(**latent), mlp=sb.model.MLP_RELU_GLU), base["layers"][1]]
    m = sb.Model(ctx, dict(base, n_layers=3, layers=layers))
    for k, v in w.items():
        m.set_tensor(k.replace("l1.", "l2.") if k.startswith("l1.") else k, MM.bf16_bits(v))
    for k, v in lw.items():
        m.set_tensor("l1." + k, MM.bf16_bits(v))
    t = rng.integers(0, vocab, 120).astype(np.int32)
    f = {k: v.astype(np.float64) for k, v in {**w, **{"x." + k: v for k, v in lw.items()}}.items()}
    pos, eps = np.arange(120), cfg["norm"]["eps"]
    x = P.layer(f["embed"][t], "l0.", cfg["layers"][0], cfg, f)
    h = P.rms(x, eps) * f["x.norm1"]
    mix = dict(latent, rot={"base": 500.0}, mask={"size": 20})
    kept = PL.latent_keys(h, f["x.mix.dkv"], f["x.mix.dkv.norm"], eps, 32, pos, 500.0)
    y = PL.latent_attention(h, *kept, mix, f["x.mix.q"], f["x.mix.uk"], f["x.mix.uv"], f["x.mix.o"], pos) * f["x.ls1"]
    x = x + cfg["residual_mult"] * (y + P.feed_forward(h, f["x.mlp.gate"], f["x.mlp.up"], f["x.mlp.down"]) * f["x.ls2"])
    x = P.layer(x, "l1.", cfg["layers"][1], cfg, f)
    want = P.rms(x, eps) * f["final.norm"] @ f["head"].T * cfg["logit_scale"]
    kv = m.new_cache(1, 160)
    for sizes in ([120], [50] + [1] * 40 + [30]):
        kv.reset()
        check(portions(kv, t, sizes), want, dtype, sizes[:2])
    kv.dispose(), m.dispose()
