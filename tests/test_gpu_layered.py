"""Models described layer by layer on the GPU against the plain implementation (plain_layered.py, float64):
whole prompts, prompts in portions, token-by-token decoding, unequal batches, caches used again, window and
tile edges, greedy generation, in bf16 and in fp32.

The error of a row of logits is the root mean square of its difference (mean taken off) over that of the
reference row. fp32 rounding alone gives about 1e-6, bf16 about 5e-3 per layer of these models."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import layered_models as LM
import plain_layered as P
import strict_b200 as sb
from strict_b200 import checkpoint, generate
from strict_b200 import native as N
from strict_b200.kernel import DeviceVariable as DV

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
LIMIT = {sb.FP32: 3e-5, sb.BF16: 3e-2}
DTYPES = [sb.FP32, sb.BF16]
dtypes = pytest.mark.parametrize("dtype", DTYPES, ids=["fp32", "bf16"])
_weights, _plain = {}, {}


def weights_of(name, gain=1.0):
    return _weights.setdefault((name, gain), LM.weights(LM.CONFIGS[name], 11, gain))


def tokens_of(name, n, seed=5):
    return np.random.default_rng(seed).integers(0, LM.CONFIGS[name]["vocab"], n).astype(np.int32)


def plain(name, tokens, gain=1.0):
    key = (name, gain, tuple(int(t) for t in tokens))
    if key not in _plain:
        _plain[key] = P.forward(LM.CONFIGS[name], weights_of(name, gain), tokens)
    return _plain[key]


def make(ctx, cfg, w, dtype, max_pos=2048):
    m = sb.Model(ctx, checkpoint.ARCHITECTURES["Kipatar"](cfg, max_pos, dtype))
    for k, v in w.items():
        m.set_tensor(k, LM.bf16_bits(v))
    return m


@pytest.fixture(scope="module")
def models(ctx):
    made = {}

    def get(name, dtype, gain=1.0):
        if (name, dtype, gain) not in made:
            made[name, dtype, gain] = make(ctx, LM.CONFIGS[name], weights_of(name, gain), dtype)
        return made[name, dtype, gain]

    yield get
    for m in made.values():
        m.dispose()


def row_errors(got, want):
    d = np.asarray(got, np.float64) - want
    d -= d.mean(-1, keepdims=True)
    c = want - want.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1) / (c * c).mean(-1))


def check(got, want, dtype, what=""):
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
@pytest.mark.parametrize("M,d,groups,splits", [(5, 96, 3, 0), (3, 90, 5, 2), (4, 2048, 1, 3), (300, 4096, 2, 0), (33, 4096, 1, 8), (2, 8200, 1, 0), (1, 7, 7, 1)])
def test_group_norm(ctx, rng, M, d, groups, splits):
    x, part = rng.standard_normal((M, d)).astype(np.float32), rng.standard_normal((max(splits, 1), M, d)).astype(np.float32)
    g1, g2 = rng.standard_normal((2, d)).astype(np.float32)
    total = x.astype(np.float64) + (part.sum(0, dtype=np.float64) if splits else 0)
    for f32 in (0, 1):
        dx, dp, d1, d2 = (DV.of(ctx, a) for a in (x, part, g1, g2))
        t = np.float32 if f32 else np.uint16
        y1, y2 = DV(ctx, M * d, t), DV(ctx, M * d, t)
        N.check(N.lib().strictb200_group_rmsnorm(ctx.h, dx.p, dp.p if splits else None, max(splits, 1), d1.p, d2.p, 1e-4, groups, M, d, y1.p, y2.p, f32))
        assert np.allclose(dx.to_host().reshape(M, d), total, rtol=1e-6, atol=1e-5)
        for y, g in ((y1, g1), (y2, g2)):
            got = y.to_host().reshape(M, d)
            got = got if f32 else (got.astype(np.uint32) << 16).view(np.float32)
            want = P.group_rms_norm(total, g.astype(np.float64), 1e-4, groups)
            assert np.allclose(got, want, rtol=2e-5 if f32 else 5e-3, atol=1e-5)
        for v in (dx, dp, d1, d2, y1, y2):
            v.free()


def test_xielu(ctx):
    x = np.concatenate([np.linspace(-30, 30, 999), [0.0, 1e-6, -1e-6, -1e-3]]).astype(np.float32)
    dx, dy = DV.of(ctx, x), DV(ctx, len(x))
    for p, q in ((0.4, -1.3), (-3.0, 2.0)):
        N.check(N.lib().strictb200_xielu(ctx.h, dx.p, len(x), p, q, dy.p))
        assert np.allclose(dy.to_host(), P.xielu(x.astype(np.float64), np.float32(p), np.float32(q)), rtol=3e-6, atol=3e-6)
    dx.free(), dy.free()


@pytest.mark.parametrize("M,Nn,K", [(1, 40, 8), (7, 300, 72), (33, 128, 520), (100, 257, 136), (129, 256, 64), (300, 520, 328), (513, 1024, 1000)])
def test_gemm_bf16(ctx, rng, M, Nn, K):
    x, w = LM.round_bf16(rng.standard_normal((M, K))), LM.round_bf16(rng.standard_normal((Nn, K)))
    dx, dw, dy = DV.of(ctx, LM.bf16_bits(x)), DV.of(ctx, LM.bf16_bits(w)), DV(ctx, M * Nn)
    want = x.astype(np.float64) @ w.T.astype(np.float64)
    N.check(N.lib().strictb200_gemm_bf16(ctx.h, M, Nn, K, dx.p, dw.p, dy.p, 1))
    assert np.allclose(dy.to_host().reshape(M, Nn), want, rtol=1e-4, atol=1e-4 * np.sqrt(K))
    db = DV(ctx, M * Nn, np.uint16)
    N.check(N.lib().strictb200_gemm_bf16(ctx.h, M, Nn, K, dx.p, dw.p, db.p, 0))
    assert np.allclose((db.to_host().astype(np.uint32) << 16).view(np.float32).reshape(M, Nn), want, rtol=5e-3, atol=1e-2)
    for v in (dx, dw, dy, db):
        v.free()
    with pytest.raises(ValueError):
        N.check(N.lib().strictb200_gemm_bf16(ctx.h, 4, 8, 12, dx.p, dw.p, dy.p, 1))


ONE = {  # one part of the layer at a time
    "attention only": LM.config([LM.entry(3, 16, 4, 24, 32, 9, None)], 64, 50, 2),
    "rotation only": LM.config([LM.entry(2, 1, 64, 16, 32, 100, None, base=40.0)], 64, 50, 2),
    "hardly any rotation": LM.config([LM.entry(2, 48, 2, 16, 32, 100, None)], 64, 50, 2),
    "window of one": LM.config([LM.entry(2, 16, 8, 16, 32, 1, 24)], 64, 50, 1),
    "a scale": LM.config([LM.entry(2, 16, 8, 16, 32, 50, None, scale=0.9)], 64, 50, 1),
    "shared latents": LM.config([LM.entry(2, 16, 8, 16, 32, 5, None), LM.entry(4, 8, 8, 40, 32, 60, None, kv_from=0)], 64, 50, 1),
}


@dtypes
@pytest.mark.parametrize("what", list(ONE))
def test_one_mechanism(ctx, what, dtype):
    cfg = ONE[what]
    w = LM.weights(cfg, 2, 1.0 if what == "a scale" else 3.0)
    t = np.random.default_rng(8).integers(0, cfg["vocab"], 100).astype(np.int32)
    want = P.forward(cfg, w, t)
    m = make(ctx, cfg, w, dtype, 128)
    kv = m.new_cache(1, 128)
    check(portions(kv, t, [100]), want, dtype, "prompt")
    kv.reset()
    check(portions(kv, t, [70] + [1] * 30), want, dtype, "decode")
    kv.dispose(), m.dispose()


# ------------------------------------------------------------------ prompts, decoding, portions
@dtypes
@pytest.mark.parametrize("name,n", [("shared", 330), ("ragged", 150), ("wide", 120), ("many-heads", 300), ("no-window", 290), ("cluster-norm", 70)])
def test_whole_prompts(models, name, n, dtype):
    t = tokens_of(name, n)
    m = models(name, dtype)
    kv = m.new_cache(1, n)
    nxt, logits = kv.prefill_rows([t], [range(n)])
    check(logits, plain(name, t), dtype)
    assert nxt[0] == logits[-1].argmax()
    kv.dispose()


@dtypes
@pytest.mark.parametrize("name,n,first", [("shared", 330, 1), ("ragged", 150, 1), ("wide", 60, 20), ("many-heads", 300, 190), ("no-window", 140, 1), ("cluster-norm", 70, 3)])
def test_decoding_token_by_token(models, name, n, first, dtype):
    """Past every window, 64-key tiles and the plan's growth; the same positions as in the prompt."""
    t = tokens_of(name, 330 if name == "shared" else n)[:n]
    kv = models(name, dtype).new_cache(1, n)
    check(portions(kv, t, [first] + [1] * (n - first)), plain(name, t), dtype)
    assert kv.lens().tolist() == [n]
    kv.dispose()


SIZES = {"pairs": [2] * 60, "threes": [3] * 40, "mixed": [5, 1, 2, 1, 1, 31, 2, 64, 2, 1, 10], "tile edges": [63, 2, 55], "tile": [64, 56], "two and rest": [2, 118]}


@dtypes
@pytest.mark.parametrize("sizes", list(SIZES))
@pytest.mark.parametrize("name", ["shared", "ragged", "no-window"])
def test_portions(models, name, sizes, dtype):
    t = tokens_of(name, 120)
    kv = models(name, dtype).new_cache(1, 120)
    check(portions(kv, t, SIZES[sizes]), plain(name, t), dtype)
    kv.dispose()


@pytest.mark.parametrize("name", ["wide", "many-heads"])
def test_portions_of_wide_models(models, name):
    t = tokens_of(name, 300 if name == "many-heads" else 120)
    kv = models(name, sb.BF16).new_cache(1, len(t))
    check(portions(kv, t, [2, 61, 2, 1, len(t) - 66]), plain(name, t), sb.BF16)
    kv.dispose()


@dtypes
def test_batches_of_unequal_requests(ctx, models, dtype):
    name, lens, n = "shared", [130, 1, 64, 65, 7, 200], 12
    m = models(name, dtype)
    prompts = [tokens_of(name, k, 20 + k) for k in lens]
    more = np.random.default_rng(3).integers(0, LM.CONFIGS[name]["vocab"], (n, len(lens))).astype(np.int32)
    want = [plain(name, np.concatenate([p, more[:, b]])) for b, p in enumerate(prompts)]
    tok = np.zeros((len(lens), max(lens)), np.int32)
    for row, p in zip(tok, prompts):
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
            tail = [tokens_of(name, k, 70 + k) for k in (3, 2, 40, 1, 9, 2)]
            pad = np.zeros((len(lens), 40), np.int32)
            for row, p in zip(pad, tail):
                row[:len(p)] = p
            _, logits = kv.prefill(pad, [len(p) for p in tail], want_logits=True)
            check(logits, np.stack([plain(name, np.concatenate([p, more[:, b], q]))[-1] for b, (p, q) in enumerate(zip(prompts, tail))]), dtype, "second portion")
            kv.dispose()
    finally:
        ctx.set_option("prefill_chunk", 16384)


@pytest.mark.parametrize("B", [40, 130, 260])
def test_many_sequences(models, B):
    """Decode batches of more than one token group, more than 128 and more than 256 rows, over different lengths."""
    name = "ragged"
    lens = np.array([1 + (7 * b) % 23 for b in range(B)], np.int32)
    tok = np.stack([tokens_of(name, 24, b % 9) for b in range(B)])
    kv = models(name, sb.BF16).new_cache(B, 32)
    kv.prefill(tok, lens)
    nxt, logits = kv.decode_step(tok[np.arange(B), lens], want_logits=True)
    check(logits, np.stack([plain(name, tok[b])[lens[b]] for b in range(B)]), sb.BF16)
    assert np.array_equal(nxt, logits.argmax(1))
    kv.dispose()


@dtypes
def test_a_cache_used_again(models, dtype):
    name = "shared"
    m = models(name, dtype)
    t, other = tokens_of(name, 90), tokens_of(name, 200, 99)
    fresh = m.new_cache(1, 256)
    want = portions(fresh, t, [50, 2, 1, 30] + [1] * 7)
    used = m.new_cache(1, 256)
    portions(used, other, [150] + [1] * 50)
    used.reset()
    got = portions(used, t, [50, 2, 1, 30] + [1] * 7)
    assert np.array_equal(got, want)
    check(got, plain(name, t), dtype)
    # the place in a batch does not matter either
    three = m.new_cache(3, 256)
    three.prefill(np.stack([other[:60], t[:60], other[60:120]]))
    logits = [three.decode_step([0, t[i], 1], want_logits=True)[1][1] for i in range(60, 90)]
    check(np.stack(logits), plain(name, t)[60:], dtype)
    for kv in (fresh, used, three):
        kv.dispose()


# ------------------------------------------------------------------ keys that stand out
def edge_case(window):
    """One attention layer in which one token's key stands out for one query token, whatever the distance: the scores of the
    pair come from the unrotated part. Returns config, weights, the pair (query id, key id)."""
    cfg = LM.config([LM.entry(2, 32, 8, 32, 48, window, None)], 96, 40, 2)
    w = LM.weights(cfg, 21, 2.0)
    m = cfg["layers"][0]["mixer"]
    h = P.group_rms_norm(w["embed"].astype(np.float64), w["l0.norm1"], cfg["norm"]["eps"], 2)
    c, _ = P.latent_keys(h, w["l0.mix.dkv"], w["l0.mix.dkv.norm"], cfg["norm"]["eps"], 48, np.zeros(40), m["rot"]["base"])
    q = (h @ w["l0.mix.q"].T.astype(np.float64)).reshape(40, 2, 40)[:, :, :32]
    k = (c @ w["l0.mix.uk"].T.astype(np.float64)).reshape(40, 2, 32)
    s = np.einsum("ahd,bhd->ab", q, k)
    a, b = np.unravel_index(s.argmax(), s.shape)
    w["l0.mix.q"] = LM.round_bf16(w["l0.mix.q"] * np.float32(25.0 / s.max() / m["scale"]))
    return cfg, w, int(a), int(b)


@dtypes
@pytest.mark.parametrize("window", [2, 5, 63, 64, 65, 128, 200])
def test_keys_just_inside_and_just_outside_the_window(ctx, window, dtype):
    cfg, w, ask, key = edge_case(window)
    filler = [t for t in range(40) if t not in (ask, key)]
    rng = np.random.default_rng(window)
    n = window + 150
    m = make(ctx, cfg, w, dtype, 512)
    kv = m.new_cache(1, n + 1)
    for at in (0, 1, 62, 63, 64, 100):  # where the key lies: the first tokens, tile borders, anywhere
        for distance in (window - 1, window):
            t = rng.choice(filler, at + distance + 3).astype(np.int32)
            t[at], t[at + distance] = key, ask
            want = P.forward(cfg, w, t)
            row = at + distance
            # the test is sharp: a window one off moves the row by far more than the limit
            off = json.loads(json.dumps(cfg))
            off["layers"][0]["mixer"]["mask"]["size"] = window + (1 if distance == window else -1)
            assert row_errors(P.forward(off, w, t), want)[row] > 5 * LIMIT[dtype]
            for sizes in ([len(t)], [row] + [1] * 3 if row else [1, 1, 1], [max(1, row - 1), 2, 2] if row > 1 else [len(t)]):
                kv.reset()
                check(portions(kv, t, sizes), want, dtype, (at, distance, sizes))
    kv.dispose(), m.dispose()


@dtypes
@pytest.mark.parametrize("name", ["shared", "no-window", "many-heads"])
def test_peaked_scores(models, name, dtype):
    """Scores spread widely enough for the softmax to follow a few keys; far keys then weigh as much as near ones."""
    gain = 3.0
    n = 260
    t = tokens_of(name, n, 31)
    want = plain(name, t, gain)
    m = models(name, dtype, gain)
    kv = m.new_cache(1, n)
    limit = LIMIT[dtype] * (3 if dtype == sb.BF16 else 2)  # the softmax passes rounding of the scores on, amplified
    for sizes in ([n], [200] + [1] * 60, [100, 2, 63, 95]):
        kv.reset()
        e = row_errors(portions(kv, t, sizes), want)
        assert e.max() <= limit and np.median(e) <= LIMIT[dtype], (sizes, int(e.argmax()), e.max(), np.median(e))
    kv.dispose()


@dtypes
def test_long_decoding(models, dtype):
    name, n = "ragged", 700
    t = tokens_of(name, n, 44)
    kv = models(name, dtype).new_cache(1, n)
    got = portions(kv, t, [5] + [1] * (n - 5))
    check(got, plain(name, t), dtype)
    kv.dispose()


# ------------------------------------------------------------------ generation, folders, replay
@dtypes
def test_greedy_generation(models, dtype):
    name, new = "shared", 24
    prompts = [tokens_of(name, k, 50 + k).tolist() for k in (9, 1, 70)]
    got = generate.greedy(models(name, dtype), prompts, new)
    for ids, p in zip(got, prompts):
        picks, margins = P.greedy(LM.CONFIGS[name], weights_of(name), p, new)
        for s in range(new):
            if ids[s] != picks[s]:
                assert margins[s] < (1e-3 if dtype == sb.FP32 else 0.25), (s, margins[s])  # a near tie: the paths part here
                break


def test_plain_launches_and_graph_agree(models, ctx):
    m = models("shared", sb.BF16)
    t = tokens_of("shared", 100)
    out = []
    for graph in (True, False):
        m.set_graph(graph)
        kv = m.new_cache(1, 100)
        out.append(portions(kv, t, [60] + [1] * 40))
        kv.dispose()
    m.set_graph(True)
    assert np.array_equal(out[0], out[1])


def test_an_activation_set_after_recording_takes_effect(ctx):
    cfg = ONE["window of one"]
    w = LM.weights(cfg, 6)
    m = make(ctx, cfg, w, sb.BF16, 64)
    t = np.arange(20, dtype=np.int32)
    kv = m.new_cache(1, 64)
    portions(kv, t, [5] + [1] * 15)
    w["l0.mlp.act"] = np.array([2.0, -2.0], np.float32)
    m.set_tensor("l0.mlp.act", w["l0.mlp.act"])
    kv.reset()
    check(portions(kv, t, [5] + [1] * 15), P.forward(cfg, w, t), sb.BF16)
    kv.dispose(), m.dispose()


@dtypes
def test_tensors_round_trip(models, dtype):
    m = models("ragged", dtype)
    for k, v in weights_of("ragged").items():
        assert np.array_equal(m.get_tensor(k, np.float32, v.size).reshape(v.shape), v), k
        assert np.array_equal(m.get_tensor(k, np.uint16, v.size).reshape(v.shape), LM.bf16_bits(v)), k
    for bad in ("l1.mlp.up", "l2.mix.dkv", "l9.norm1", "l0.mix", "norm", "l.norm1"):
        with pytest.raises(ValueError):
            m.set_tensor(bad, np.zeros(4, np.float32))
    with pytest.raises(ValueError):
        m.set_tensor("embed", np.zeros(3, np.float32))


def test_configurations_that_are_refused(ctx):
    good = checkpoint.ARCHITECTURES["Kipatar"](LM.CONFIGS["shared"], 64, sb.BF16)
    for layer, key, value in ((1, "kv_from", 1), (1, "kv_from", 3), (3, "kv_from", 1), (1, "kv_rank", 72), (1, "rot_base", 1.0), (0, "rot_dim", 7), (0, "heads", 0)):
        bad = json.loads(json.dumps(good))
        bad["layers"][layer][key] = value
        with pytest.raises(ValueError):
            sb.Model(ctx, bad)
    for key, value, error in (("norm_groups", 5, ValueError), ("dtype", 3, ValueError)):
        with pytest.raises(error):
            sb.Model(ctx, dict(good, **{key: value}))
    bad = json.loads(json.dumps(good))
    bad["layers"][0]["mixer"] = 9
    with pytest.raises(NotImplementedError):
        sb.Model(ctx, bad)


def test_folder_and_replay(tmp_path):
    """bin/trace_run in a process of its own: portions, single tokens, wanted places, a second request after the first."""
    name = "ragged"
    cfg, w = LM.CONFIGS[name], weights_of(name)
    LM.write_folder(tmp_path, cfg, w)
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
        assert [x for x in p.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(len(plan))]
        for i, (r, lo, n, want) in enumerate(plan):
            path = out / f"{i}.f32"
            assert path.exists() == bool(want)
            if want:
                got = np.fromfile(path, "<f4").reshape(len(want), -1)
                check(got, plain(name, seqs[r])[[lo + k for k in want]], dtype, i)
    p = subprocess.run([sys.executable, "-m", "strict_b200.generate", "--model", str(tmp_path), "--prompt", "1,2,3", "--prompt", "4", "--new", "5", "--dtype", "float32"],
                       capture_output=True, text=True, timeout=600, cwd=ROOT)
    assert p.returncode == 0, p.stderr[-2000:]
    ids = [[int(x) for x in line.split(",")] for line in p.stdout.split()]
    assert [len(x) for x in ids] == [5, 5] and ids[0] == P.greedy(cfg, w, [1, 2, 3], 5)[0]


# ------------------------------------------------------------------ rows of the other models' prompts
@pytest.mark.parametrize("cfg", [dict(arch=1, n_layers=2, d_model=256, n_q_heads=4, n_kv_heads=2, head_dim=128, d_ff=512, vocab=1024, max_pos=128, tied=0, eps=1e-6, rope_theta=1e6),
                                 dict(arch=0, n_layers=2, d_model=128, n_q_heads=2, n_kv_heads=2, head_dim=64, d_ff=512, vocab=512, max_pos=64, tied=1, eps=1e-5, rope_theta=0.0)],
                         ids=["qwen", "gpt2"])
def test_wanted_rows_of_other_models(ctx, cfg):
    m = sb.Model(ctx, cfg).init_random(9)
    t = np.random.default_rng(0).integers(0, cfg["vocab"], (2, 30)).astype(np.int32)
    kv = m.new_cache(2, 64)
    nxt, rows = kv.prefill_rows(t, [[4, 29], [0]], [30, 21])
    for r, (b, n) in enumerate(((0, 5), (0, 30), (1, 1))):
        kv.reset()
        _, want = kv.prefill(t[:, :n], want_logits=True)
        assert np.abs(rows[r] - want[b]).max() <= 2e-2
    kv.reset()
    assert np.array_equal(kv.prefill(t, [30, 21])[0], nxt)
    with pytest.raises(ValueError):
        kv.prefill_rows(t, [[30], []])
    kv.dispose(), m.dispose()
