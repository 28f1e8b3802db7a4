"""The Zetalorn decoder through its executor, scheduler and command line against the plain forward pass of
zetalorn_reference.py: a packed step must give every sequence the logits of its whole history run alone, however the
history was cut, batched or placed."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import stack_harness
import zetalorn_reference as R
from logismos_b200.embed import ComputeError, InputTooLong
from logismos_b200.generate import generate, sampling_chain
from logismos_b200.registry import Limits, load_model
from logismos_b200.replay import Replay
from logismos_b200.zetalorn import ZetalornModel, parse_config
from stack_harness import TOLS, greedy_reference, tokens
from zetalorn_weights import CONFIGS, attention, config, left, moe, pack, parallel, right, rotation, weights

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BOTH = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
EVERY = pytest.mark.parametrize("name", sorted(CONFIGS))
BEACON, SEEKER, FILLER = 3, 4, 5       # marked tokens; others are drawn from FILLER on


def Harness(cfg, w, dtype, **kw):
    return stack_harness.Harness(ZetalornModel, pack, R.forward, cfg, w, dtype, **kw)


def feed(h, sid, prompt, cuts):
    """A history fed in portions (empty ones are left out), then given back."""
    h.known(sid, prompt)
    at = 0
    for c in cuts:
        if c:
            h.run([(sid, prompt[at:at + c])])
        at += c
    assert at == len(prompt)
    h.drop(sid)


@BOTH
@EVERY
def test_every_layer_of_every_pass(name, dtype):
    cfg, w = CONFIGS[name], weights(name, 10)
    h = Harness(cfg, w, dtype, keep_layers=True)
    prompt = tokens(np.random.default_rng(0), cfg, 75)
    layers = []
    R.forward(cfg, w, prompt, layers)
    assert len(layers) == h.model.cfg["n_layers"]
    at = 0
    for n in (70, 1, 1, 2, 1):
        h.run([("a", prompt[at:at + n])])
        assert np.array_equal(h.model.snapshot(0), w["embed"][prompt[at:at + n]].astype(np.float32))
        for i, x in enumerate(layers):
            h.compare(h.model.snapshot(i + 1), x[at:at + n], (i, at), x)
        at += n
    h.close()


@BOTH
@EVERY
def test_prompt_portions_and_decoding_agree(name, dtype):
    """One token, a whole prompt, the same prompt token by token, and cut into portions down to two tokens, at page, window,
    block and chunk borders; pages and slots are given back and used again in between."""
    cfg = CONFIGS[name]
    h = Harness(cfg, weights(name, 11), dtype)
    rng = np.random.default_rng(1)
    h.run([("one", tokens(rng, cfg, 1))])
    prompt = tokens(rng, cfg, 200)
    whole = h.run([("w", prompt)])
    h.drop("one")
    for t in range(45):
        z = h.run([("d", prompt[t:t + 1])], check=False)
        h.compare(z, whole[t:t + 1], ("decoded against prompt", t), whole, factor=2.0)   # both sides are rounded
    h.drop("w")
    for k, cuts in enumerate(([2] * 10 + [180], [15, 1, 1, 16, 17, 3, 147], [63, 2, 64, 21, 50], [128, 2, 70], [149, 1, 2, 48], [1, 2, 3, 194], [39, 1, 40, 2, 39, 1, 78])):
        feed(h, k, prompt, cuts)
    h.close()


@BOTH
@EVERY
def test_mixed_batches_of_unequal_requests(name, dtype):
    cfg = CONFIGS[name]
    h = Harness(cfg, weights(name, 12), dtype)
    rng = np.random.default_rng(2)
    T = lambda n: tokens(rng, cfg, n)
    h.run([("a", T(70)), ("b", T(1)), ("c", T(2)), ("d", T(33))])
    h.run([("c", T(1)), ("e", T(129)), ("a", T(1)), ("d", T(2))])          # b is left out and goes on later
    h.run([("b", T(1)), ("a", T(1)), ("c", T(1)), ("e", T(1))])
    h.drop("a"); h.drop("d")
    h.run([("f", T(50)), ("b", T(17)), ("g", T(3)), ("e", T(5)), ("c", T(1))])  # pages and slots of a and d again
    h.run([("g", T(2)), ("f", T(1)), ("b", T(1))])
    for _ in range(6):
        h.run([("e", T(1)), ("g", T(1)), ("b", T(1)), ("f", T(1)), ("c", T(1))])
    h.close()


# ---- marked keys: one score stands out ----------------------------------------------------------------

def mark(w, q, k, rot, maps=1):
    """BEACON and SEEKER have a feature each that no other token has. The first head's unrotated channels (of its first map) answer
    to nothing else, so that the beacon's key decides the seeker's output wherever it stands in sight; another key scores
    nothing there, and a pooled block of the beacon its share."""
    w["embed"][:, :2] = 0.0
    w["embed"][BEACON, 0] = w["embed"][SEEKER, 1] = 6.0
    dim = w[q + ".norm"].size
    free = slice(rot["dims"], dim)
    signs = np.where(np.arange(dim - rot["dims"]) % 3 == 0, -1.0, 1.0)
    for name, feature in ((q, 1), (k, 0)):
        m = w[name]
        for head in range(m.shape[0] // dim):
            if maps == 1 or head % 2 == 0:
                m[head * dim + rot["dims"]:(head + 1) * dim] = 0.0
                m[head * dim + rot["dims"]:(head + 1) * dim, feature] = 4.0 * signs
        w[name + ".norm"][free] = 2.0
    return w


def pooled_model(size, pool):
    rot = rotation(16, 1e4)
    cfg = config(120, 64, [parallel(left(2, 1, 32, 32, size, pool, rot, scale=0.5), right(16, 16, (0.5,)))], eps=1e-6)
    w = mark(R.random_weights(cfg, 7), "l0.mix.left.q", "l0.mix.left.k", rot)
    w["l0.mix.right.out"][:] = 0.0     # the other branch remembers everything: it stays out
    w["l0.rg1.b"][:] = 2.0
    return cfg, w


def chunk_model(size):
    rot = rotation(16, 1e4, 2.0)
    cfg = config(120, 64, [attention(2, 1, 32, 40, size, rot, 0.3, scale=0.5)], eps=1e-6)
    w = mark(R.random_weights(cfg, 7), "l0.mix.q", "l0.mix.k", rot, maps=2)
    w["l0.rg1.b"][:] = 2.0
    return cfg, w


def moved(cfg, w, prompt, place, at=-1):
    """How far the logits of a position move with another token at `place`."""
    other = np.array(prompt)
    other[place] = FILLER + 40
    a, b = R.forward(cfg, w, prompt), R.forward(cfg, w, other)
    return np.sqrt(np.mean((a[at] - b[at]) ** 2)) / np.sqrt(np.mean(a ** 2))


def marked(rng, n, place, cfg):
    p = rng.integers(FILLER, cfg["vocab"], n)
    p[place], p[-1] = BEACON, SEEKER
    return p


def check_place(h, cfg, w, p, place, seen, sid):
    m = moved(cfg, w, p, place)
    assert (m > 3 * TOLS["bfloat16"]) == seen and (seen or m == 0.0), (sid, m)
    n = len(p)
    for k, cuts in enumerate(([n], [n - 1, 1], [n - 2, 2], [place + 1, n - place - 1], [place, 1, n - place - 1], [max(0, n - 9), min(n, 9) - 1, 1])):
        feed(h, (sid, k), p, cuts)


@BOTH
@pytest.mark.parametrize("size,pool", [(20, 4), (64, 8), (130, 5), (16, 16), (7, 20), (33, 1), (1, 3)])
def test_window_and_block_edges(size, pool, dtype):
    """The marked key just inside and just outside the window, in a block that is just seen and one that is not yet, found by a
    prompt and by a decoded token; portions that end around it."""
    cfg, w = pooled_model(size, pool)
    h = Harness(cfg, w, dtype, pool_tokens=2048, step_tokens=1400)
    rng = np.random.default_rng(size)
    b = 300 // pool
    first, last = b * pool, b * pool + pool - 1
    cases = [("window_in", first, first + size, True)]                  # the seeker at first + size - 1
    if pool > 1:
        cases += [("window_out", first, first + size + 1, pool == 1), ("pool_out", first, last + size, False)]
        cases += [("pool_out, middle", first + pool // 2, last + size, first + pool // 2 > last - 1)]
    cases += [("pool_in, first", first, last + size + 1, True), ("pool_in, last", last, last + size + 1, True), ("pool_in, later", first + pool // 2, last + size + 18, True)]
    for what, place, n, seen in cases:
        if size == 1 and place == n - 1:
            continue                                                     # the seeker's own place
        check_place(h, cfg, w, marked(rng, n, place, cfg), place, seen, what)
    h.close()


@BOTH
@pytest.mark.parametrize("size", [20, 64, 130, 3])
def test_chunk_edges(size, dtype):
    """The marked key as the first of the seeker's chunk and as the last of the one before."""
    cfg, w = chunk_model(size)
    h = Harness(cfg, w, dtype, pool_tokens=2048, step_tokens=1400)
    rng = np.random.default_rng(size)
    start = -(-300 // size) * size
    for what, place, n, seen in (("first", start, start + size, True), ("next", start, start + 2, True), ("before", start - 1, start + 1, False), ("before, far", start - 1, start + size, False),
                                 ("the start", 0, size, True), ("the start, gone", 0, size + 1, False), ("last", start - 2, start, True)):
        check_place(h, cfg, w, marked(rng, n, place, cfg), place, seen, what)
    h.close()


@BOTH
def test_far_blocks_among_hundreds(dtype):
    """A pooled block a thousand tokens back, at page, table and tile borders."""
    cfg, w = pooled_model(40, 4)
    h = Harness(cfg, w, dtype, pool_tokens=2048, step_tokens=1400)
    rng = np.random.default_rng(9)
    for place in (0, 1, 15, 16, 63, 64, 127, 511, 512, 513):
        p = marked(rng, 1300, place, cfg)
        assert moved(cfg, w, p, place) > 2 * TOLS["bfloat16"]
        feed(h, place, p, [1299, 1] if place % 2 else [700, 3, 596, 1])
    feed(h, "whole", p, [1300])
    h.close()


@BOTH
def test_windows_pass_over_decoded_tokens(dtype):
    """The marked key is decoded; the window passes it, its block is not seen yet, and then is, one token at a time."""
    for cfg, w in (pooled_model(18, 6), pooled_model(5, 20), chunk_model(24)):
        h = Harness(cfg, w, dtype)
        p = np.random.default_rng(4).integers(FILLER, cfg["vocab"], 110)
        p[40] = BEACON
        p[41:] = SEEKER
        feed(h, "a", p, [33] + [1] * 77)
        h.close()


def recurrence_model():
    """Decays near one, and a token whose key is a hundred times the others': its trace decides what follows."""
    cfg = config(60, 48, [parallel(left(2, 1, 16, 16, 8, 4, rotation(8)), right(24, 20, (0.9995, 0.9999)))], eps=1e-6)
    w = R.random_weights(cfg, 8)
    w["l0.mix.left.out"][:] = 0.0
    w["embed"][:, 0] = 0.0
    w["embed"][BEACON, 0] = 6.0
    k = w["l0.mix.right.k"]
    w["l0.mix.right.k"] = R.bf16(np.concatenate([np.abs(8.0 * np.sign(k[:, :1])), 0.04 * k[:, 1:]], axis=1))
    w["l0.rg1.b"][:] = 2.0
    return cfg, w


@BOTH
def test_far_tokens_of_the_recurrence(dtype):
    """The state must pass through chunks, cuts and slots, over a thousand tokens and from any place of a chunk."""
    cfg, w = recurrence_model()
    h = Harness(cfg, w, dtype, pool_tokens=2048, step_tokens=1400)
    rng = np.random.default_rng(3)
    prompt = rng.integers(FILLER, cfg["vocab"], 1200)
    prompt[20] = BEACON
    assert moved(cfg, w, prompt, 20) > 3 * TOLS["bfloat16"]
    for k, cuts in enumerate(([1200], [20, 63, 65, 1, 1, 2, 1048], [1196, 1, 1, 1, 1])):
        feed(h, k, prompt, cuts)
    for first in (0, 15, 16, 47, 63, 64, 65, 127):
        p = rng.integers(FILLER, cfg["vocab"], 150)
        p[first] = BEACON
        feed(h, first, p, [first + 2, 147 - first, 1])
    h.close()


@BOTH
def test_long_prompts_whose_recurrences_run_in_segments(dtype):
    """One long prompt beside short ones and decoded tokens, then portions that end inside a segment."""
    cfg = config(90, 48, [parallel(left(2, 1, 16, 16, 40, 8, rotation(8)), right(24, 20, (0.9, 0.999))), attention(2, 1, 16, 24, 100, rotation(8), 0.3)])
    h = Harness(cfg, R.random_weights(cfg, 23), dtype, pool_tokens=4096, step_tokens=2600)
    rng = np.random.default_rng(5)
    T = lambda n: tokens(rng, cfg, n)
    h.run([("a", T(1)), ("b", T(40))])
    h.run([("long", T(1100)), ("a", T(1)), ("b", T(2)), ("c", T(700))])
    h.run([("c", T(600)), ("long", T(1)), ("a", T(3))])
    h.run([("long", T(1030)), ("c", T(1))])
    h.run([("long", T(1)), ("c", T(1)), ("a", T(1)), ("b", T(1))])
    h.close()


def test_passes_keep_their_caches_and_states_apart():
    """A model whose passes are written out as layers with equal tensors, the embedding and the steps added by hand."""
    base = [parallel(left(2, 1, 16, 16, 9, 2, rotation(8)), right(16, 16, (0.9, 0.8)), moe(4, 2, 16, 2, 1)), attention(2, 1, 8, 16, 6, rotation(8), 0.2)]
    cfg = config(70, 48, base, loop=(0, 2, 3))
    w = R.random_weights(cfg, 3)
    prompt = tokens(np.random.default_rng(4), cfg, 40)
    h = Harness(cfg, w, "float32", keep_layers=True)
    h.run([("a", prompt[:30])])
    for t in range(30, 40):
        h.run([("a", prompt[t:t + 1])])
    h.close()
    # without steps and with one pass nothing but the layers remains
    w["loop.step"] = w["loop.step"][:1] * 0.0
    zs = []
    for c in (dict(cfg, loop={"start": 0, "stop": 2, "times": 1}), {k: v for k, v in cfg.items() if k != "loop"}):
        h = Harness(c, w if "loop" in c else {k: v for k, v in w.items() if k != "loop.step"}, "float32")
        zs.append(h.run([("a", prompt)]))
        h.close()
    assert np.array_equal(zs[0], zs[1])


@BOTH
def test_long_decoding_with_reused_pages(dtype):
    cfg = CONFIGS["uneven"]
    h = Harness(cfg, weights("uneven", 21), dtype, pool_tokens=640, max_seqs=2)
    all_tokens = tokens(np.random.default_rng(3), cfg, 330)
    for turn in range(2):                      # the second turn's pages are the first's
        h.known(turn, all_tokens)
        h.run([(turn, all_tokens[:20])])
        out = [h.run([(turn, all_tokens[t:t + 1])], check=False)[0] for t in range(20, 330)]
        h.compare(np.stack(out), h.expect(turn)[20:], turn)
        h.drop(turn)
    h.close()


def test_logits_do_not_depend_on_the_batch():
    """The same tokens alone and among others, with other pages and slots: equal up to rounding."""
    for dtype, tol in (("float32", 1e-5), ("bfloat16", 3e-2)):
        cfg, w = CONFIGS["uneven"], weights("uneven", 31)
        rng = np.random.default_rng(4)
        a, b, c = (tokens(rng, cfg, n) for n in (60, 90, 3))
        got = []
        for block_seed, others in ((1, False), (2, True)):
            h = Harness(cfg, w, dtype, block_seed=block_seed)
            rest = [("b", b), ("c", c)] if others else []
            z = [h.run(rest[:1] + [("a", a[:25])] + rest[1:], check=False)]
            z = [z[0][len(b) if others else 0:][:25]]
            for t in range(25, 30):
                z.append(h.run([("a", a[t:t + 1])] + ([("c", c[:1])] if others else []), check=False)[:1])
            z.append(h.run(([("b", b[:2])] if others else []) + [("a", a[30:])], check=False)[-30:])
            got.append(np.concatenate(z))
            h.close()
        assert np.sqrt(np.mean((got[0] - got[1]) ** 2)) <= tol * np.sqrt(np.mean(got[0] ** 2))


def test_many_sequences_decode_together():
    """Steps of 20, 40 and 140 sequences: every route of the projections, the router and the experts at decode."""
    cfg, w = CONFIGS["uneven"], weights("uneven", 61)
    for n in (20, 40, 140):
        h = Harness(cfg, w, "bfloat16", pool_tokens=16 * n * 2, max_seqs=n, step_tokens=n * 9)
        h.worst = np.inf       # among so many tokens some router nearly ties
        rng = np.random.default_rng(n)
        seqs = [tokens(rng, cfg, 12) for _ in range(n)]
        h.run([(i, s[:3 + i % 6]) for i, s in enumerate(seqs)])
        for t in range(3):
            h.run([(i, s[3 + i % 6 + t:4 + i % 6 + t]) for i, s in enumerate(seqs)])
        h.close()


def test_heads_of_equal_width_on_both_sides():
    """Both output projections as one batch of short steps, and apart in larger ones and beside unequal sides."""
    layers = [parallel(left(4, 2, 64, 64, 24, 8, rotation(32, 1e4)), right(64, 128, (0.9, 0.99)), moe(8, 2, 64, 2, 1)), parallel(left(2, 1, 64, 64, 24, 8, rotation(32, 1e4)), right(64, 128, (0.9, 0.99)))]
    cfg = config(150, 128, layers)
    w = R.random_weights(cfg, 17)
    for dtype in ("float32", "bfloat16"):
        h = Harness(cfg, w, dtype, max_seqs=40)
        rng = np.random.default_rng(1)
        seqs = [tokens(rng, cfg, 8) for _ in range(36)]
        h.run([(i, s[:4]) for i, s in enumerate(seqs)])
        for lo, hi, t in ((0, 3, 4), (0, 16, 5), (0, 36, 6)):
            h.run([(i, seqs[i][len(h.hist[i]):len(h.hist[i]) + 1]) for i in range(lo, hi)])
        h.close()


# ---- through the framework's own entry points ----------------------------------------------------------

def test_greedy_generation_through_scheduler_and_command_line(tmp_path):
    """Prompts fed in chunks beside decoding sequences, more requests than slots, from a model folder."""
    cfg, w = CONFIGS["uneven"], weights("uneven", 41)
    R.write_checkpoint(tmp_path, cfg, w)
    rng = np.random.default_rng(6)
    prompts = [tokens(rng, cfg, n).tolist() for n in (40, 1, 17, 64, 2)]
    want = [greedy_reference(R.forward, cfg, w, p, 10) for p in prompts]
    assert min(m for _, m in want) > 1e-3      # no near ties: the continuation is defined
    served = load_model(str(tmp_path), Limits(192, 3, max_step_tokens=30), "float32")
    got = generate(served, prompts, 10, prefill_token_budget=24)
    served.close()
    assert got == [t for t, _ in want]
    r = subprocess.run([sys.executable, "-m", "logismos_b200.generate", "--model", str(tmp_path), "--dtype", "float32", "--max-new", "10",
                        "--max-seqs", "2", "--prefill-budget", "16"] + sum((["--prompt", ",".join(map(str, p))] for p in prompts), []),
                       capture_output=True, text=True, cwd=ROOT)
    assert r.returncode == 0, r.stderr
    assert [[int(t) for t in line.split(",")] for line in r.stdout.split()] == got


def test_sampling_chain_over_the_executors_logits(tmp_path):
    cfg = CONFIGS["narrow"]
    R.write_checkpoint(tmp_path, cfg, weights("narrow", 42))
    served = load_model(str(tmp_path), Limits(256, 4))
    prompts = [[1, 2, 3], [7], [9, 8]]
    greedy = generate(served, prompts, 8)
    assert generate(served, prompts, 8, sampling_chain(1.0, 1, 1.0, 0.0, 5)) == greedy     # top-1 is greedy
    hot = [generate(served, prompts, 8, sampling_chain(5.0, 0, 1.0, 0.0, s)) for s in (1, 1, 2)]
    assert hot[0] == hot[1] and hot[0] != hot[2] and hot[0] != greedy
    served.close()


def test_replay_of_a_schedule_from_a_folder(tmp_path):
    cfg, w = CONFIGS["large_heads"], weights("large_heads", 51)
    R.write_checkpoint(tmp_path / "m", cfg, w)
    rng = np.random.default_rng(8)
    a, b, c = (tokens(rng, cfg, n).tolist() for n in (100, 30, 64))
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:50], "want": [0, 49]}, {"id": "b", "tokens": b[:1], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[1:3], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[3:], "want": [26]}, {"id": "a", "tokens": a[50:51], "want": [0]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "c", "tokens": c, "want": [63, 5]}, {"id": "a", "tokens": a[51:], "want": [48]}], "end": ["a", "c"]}]
    za, zb, zc = (R.forward(cfg, w, t) for t in (a, b, c))
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "192"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True)
        assert r.returncode == 0, r.stderr
        assert r.stdout.split("\n")[:4] == ["done 0", "done 1", "done 2", "done 3"]
        for step, ref in ((0, [za[0], za[49]]), (2, [zb[29], za[50]]), (3, [zc[63], zc[5], za[99]])):
            z = np.fromfile(out / f"{step}.f32", "<f4").reshape(len(ref), -1)
            err = np.sqrt(np.mean((z - np.stack(ref)) ** 2, axis=1)) / np.sqrt(np.mean(za ** 2))
            assert err.max() <= TOLS[dtype]


def test_the_cache_pool_and_the_slots_are_finite(tmp_path):
    cfg = CONFIGS["narrow"]
    R.write_checkpoint(tmp_path, cfg, weights("narrow", 43))
    served = load_model(str(tmp_path), Limits(128, 2))
    r = Replay(served)
    r.step([{"id": "a", "tokens": [1] * 64, "want": []}])
    with pytest.raises(MemoryError):
        r.step([{"id": "b", "tokens": [1] * 65, "want": []}])
    r.end("a"); r.end("b")
    z = r.step([{"id": "b", "tokens": [1] * 128, "want": [127]}])          # the whole pool in one sequence
    assert np.isfinite(z).all()
    served.close()


def test_step_rejects_what_it_cannot_run():
    cfg, w = CONFIGS["narrow"], weights("narrow", 1)
    h = Harness(cfg, w, "bfloat16", pool_tokens=128, max_seqs=2, step_tokens=64)
    tab = np.arange(8, dtype=np.int32)[None]
    m = h.model
    m.step([1, 2, 3], [0], [3], tab, [0], out_rows=[])
    assert m.last_logits().shape == (0, cfg["vocab"])
    for bad in (lambda: m.step([1], [0], [1], tab, [2]), lambda: m.step([1, 2], [0, 0], [1, 1], np.concatenate([tab, tab]), [1, 1]),
                lambda: m.step([1] * 65, [0], [65], tab, [0]), lambda: m.step([1], [0], [1], tab, [0], out_rows=[1]),
                lambda: m.step([1], [0], [1], np.full_like(tab, 9), [0]), lambda: m.snapshot(0)):
        with pytest.raises(ComputeError):
            bad()
    with pytest.raises(InputTooLong):
        m.step([1], [128], [1], tab, [0])
    m.close()
    empty = {"layers": [{}], **{k: np.zeros(64 * 40, np.uint16) for k in ("embed", "head", "final_norm", "loop_step")}}
    good, side = attention(2, 1, 8, 8, 8, rotation(4)), right(8, 8, (0.5,))
    lf = lambda **kw: dict(good_left, **kw)
    good_left = left(2, 1, 8, 8, 8, 2, rotation(4))
    bad = [dict(good, mixer=dict(good["mixer"], dim=130)), dict(good, mixer=dict(good["mixer"], vdim=300)), dict(good, mixer=dict(good["mixer"], kv_heads=3)),
           dict(good, mixer=dict(good["mixer"], scale=-1.0)), dict(good, mixer=dict(good["mixer"], rot=rotation(3))), dict(good, mixer=dict(good["mixer"], rot=rotation(4, 1.0))),
           dict(good, mlp=moe(600, 2, 8, 1, 1)), dict(good, mlp=moe(8, 3, 8, 4, 1)), dict(good, mlp=moe(8, 2, 8, 3, 1)), dict(good, mlp=moe(8, 2, 8, 2, 3)),
           parallel(lf(dim=300), side), parallel(lf(scale=0.0), side), parallel(lf(mask={"size": 8, "pool": -1}), side), parallel(lf(mask={"size": 0, "pool": 2}), side),
           parallel(good_left, right(300, 8, (0.5,))), parallel(good_left, right(8, 8, (1.5,))), parallel(good_left, right(8, 8, (-0.1,))), parallel(good_left, right(8, 8, (float("nan"),)))]
    for y in bad:
        with pytest.raises(ComputeError):
            ZetalornModel(parse_config(config(64, 40, [y])), empty, 4, 4, 16, 1, 1)
    cfg = parse_config(config(64, 40, [good]))
    for change in (dict(norm=0), dict(norm=1), dict(passes=-1), dict(layers=[dict(cfg["layers"][0], **{"pass": 1})])):      # a stack or a pass that is not there
        with pytest.raises(ComputeError):
            ZetalornModel(dict(cfg, **change), empty, 4, 4, 16, 1, 1)


def test_loader_accounts_for_every_tensor(tmp_path):
    cfg, w = CONFIGS["uneven"], weights("uneven", 2)
    for name, change in (("extra", lambda d: d.update(more=np.zeros(3))), ("missing", lambda d: d.pop("l1.mix.lk2")), ("bias", lambda d: d.pop("l1.rg2.b")), ("gate", lambda d: d.pop("l2.rg1")),
                         ("norm", lambda d: d.update({"l0.norm1": np.ones(88)})), ("expert", lambda d: d.pop("l0.mlp.e4.down")), ("step", lambda d: d.pop("loop.step")),
                         ("passes", lambda d: d.update({"loop.step": d["loop.step"][:2]})), ("shape", lambda d: d.update({"l1.mix.q": d["l1.mix.q"][:-1]})),
                         ("branch", lambda d: d.pop("l0.mix.right.out")), ("correction", lambda d: d.update({"l0.mlp.correction": np.zeros(6)}))):
        d = dict(w)
        change(d)
        R.write_checkpoint(tmp_path / name, cfg, d)
        with pytest.raises((ComputeError, IOError)):
            load_model(str(tmp_path / name), Limits(64, 1))
    # a layer without a feed-forward whose norm and gate are stored all the same
    d = dict(w, **{"l2.norm2": np.asarray(1.0), "l2.rg2": w["l2.rg1"], "l2.rg2.b": w["l2.rg1.b"]})
    R.write_checkpoint(tmp_path / "idle", cfg, d)
    load_model(str(tmp_path / "idle"), Limits(64, 1)).close()
