"""The Vugedra decoder through its executor, scheduler and command line against the plain forward pass of
vugedra_reference.py: a packed step must give every sequence the logits of its whole history run alone, however the
history was cut, batched or placed."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import stack_harness
import vugedra_reference as R
from logismos_b200.embed import ComputeError, InputTooLong
from logismos_b200.generate import generate, sampling_chain
from logismos_b200.registry import Limits, load_model
from logismos_b200.replay import Replay
from logismos_b200.vugedra import VugedraModel, parse_config
from stack_harness import TOLS, greedy_reference, tokens
from vugedra_weights import CONFIGS, SIZES, again, attention, config, dense, gla, latent, moe, pack, rotation, weights

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BOTH = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
EVERY = pytest.mark.parametrize("name", sorted(CONFIGS))


def Harness(cfg, w, dtype, **kw):
    return stack_harness.Harness(VugedraModel, pack, R.forward, cfg, w, dtype, **kw)


@BOTH
@EVERY
def test_every_layer(name, dtype):
    cfg, w = CONFIGS[name], weights(name, 10)
    h = Harness(cfg, w, dtype, keep_layers=True)
    prompt = tokens(np.random.default_rng(0), cfg, 75)
    layers = []
    R.forward(cfg, w, prompt, layers)
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
    """One token, a whole prompt, the same prompt token by token, and cut into portions down to two tokens, at page, window
    and chunk borders; pages and slots are given back and used again in between."""
    cfg = CONFIGS[name]
    h = Harness(cfg, weights(name, 11), dtype)
    rng = np.random.default_rng(1)
    h.run([("one", tokens(rng, cfg, 1))])
    prompt = tokens(rng, cfg, 200)
    whole = h.run([("w", prompt)])
    h.drop("one")
    for t in range(40):
        z = h.run([("d", prompt[t:t + 1])], check=False)
        h.compare(z, whole[t:t + 1], ("decoded against prompt", t), whole, factor=2.0)   # both sides are rounded
    h.drop("w")
    for k, cuts in enumerate(([2] * 10 + [180], [15, 1, 1, 16, 17, 3, 147], [63, 2, 64, 21, 50], [128, 2, 70], [149, 1, 2, 48], [1, 2, 3, 194])):
        at = 0
        h.known(k, prompt)
        for c in cuts:
            h.run([(k, prompt[at:at + c])])
            at += c
        h.drop(k)
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
    for _ in range(4):
        h.run([("e", T(1)), ("g", T(1)), ("b", T(1)), ("f", T(1)), ("c", T(1))])
    h.close()


def _replace(q, inp, want):
    """The matrix q changed by rank one so that it maps inp to want."""
    return R.bf16(0.2 * q + np.outer(want - 0.2 * q @ inp, inp) / (inp @ inp))


@BOTH
def test_far_keys_of_latent_attention_stand_out(dtype):
    """One token's unrotated key is matched by another's query, so that a single far score decides the output: it must be
    found from any distance, across pages, chunks and cuts."""
    m = latent(2, 32, rotation(2, 1e6), 32, 48, 40, scale=0.5)
    cfg = config(120, 64, [m], eps=1e-6)
    w = R.random_weights(cfg, 5)
    beacon, seeker = 3, 4
    h = R.tanh_norm(w["embed"], w["l0.norm1.alpha"], w["l0.norm1"], w["l0.norm1.b"])
    part = {k[len("l0.mix."):]: v for k, v in w.items() if k.startswith("l0.mix.")}
    c, _ = R.latent_cache_rows(h, part, m["mixer"], 1e-6)
    k = c @ part["uk"].T
    k -= k.mean(axis=0)
    cq = R.rms_norm(h[seeker] @ part["dq"].T, part["dq.norm"], 1e-6)
    want = part["uq"] @ cq
    for a in range(2):
        rows = slice(34 * a, 34 * a + 32)
        want[rows] = 1.6 * k[beacon, 32 * a:32 * a + 32]
    w["l0.mix.uq"] = _replace(part["uq"], cq, want)
    run_far(cfg, w, dtype, beacon, seeker, lambda w, p: R.forward(cfg, w, p))


def run_far(cfg, w, dtype, beacon, seeker, forward, firsts=(1, 15, 16, 17, 39, 63, 64, 65, 127, 128, 129), gaps=(40,)):
    h = Harness(cfg, w, dtype, pool_tokens=2048, step_tokens=1400)
    rng = np.random.default_rng(9)
    filler = lambda n: rng.integers(5, cfg["vocab"], n)
    prompt = np.concatenate([filler(7), [beacon], filler(1290), [seeker], filler(3)])
    ref = forward(w, prompt)
    without = prompt.copy()
    without[7] = 60
    moved = np.sqrt(np.mean((ref[-4] - forward(w, without)[-4]) ** 2)) / np.sqrt(np.mean(ref ** 2))
    assert moved > 3 * TOLS["bfloat16"]      # the far key decides this position
    h.run([("w", prompt)])
    h.drop("w")
    for sid, cuts in (("d", [1298, 1, 1, 1, 1]), ("c", [8, 1289, 2]), ("e", [700, 3, 596, 3])):
        at = 0
        h.known(sid, prompt)
        for c in cuts:
            h.run([(sid, prompt[at:at + c])])
            at += c
        h.drop(sid)
    for first in firsts:                     # the beacon around page, table and tile borders
        for gap in gaps:
            p = np.concatenate([filler(first - 1), [beacon], filler(gap), [seeker]])
            h.run([(first, p[:-1])])
            h.run([(first, p[-1:])])
            h.drop(first)
    h.close()


def window_model(size, keep, dims=16, vocab=120, scaling=None, gain=2.0):
    """An attention layer in which the token `beacon` draws nearly all weight of `seeker` wherever it stands in sight: of the
    channels only the unrotated ones carry the match."""
    m = attention(2, 1, 32, 32, rotation(dims, 1e4, scaling), size, keep, scale=0.5)
    cfg = config(vocab, 64, [m], eps=1e-6)
    w = R.random_weights(cfg, 7)
    beacon, seeker = 3, 4
    h = R.tanh_norm(w["embed"], w["l0.norm1.alpha"], w["l0.norm1"], w["l0.norm1.b"])
    kb = w["l0.mix.k"] @ h[beacon] + w["l0.mix.k.b"]
    kb = kb / np.sqrt(np.mean(kb ** 2)) * w["l0.mix.k.norm"]
    want = np.zeros(64)
    for a in range(2):
        want[32 * a + dims:32 * a + 32] = kb[dims:]
    w["l0.mix.q.norm"] = R.bf16(np.ones(64) * gain)
    w["l0.mix.q.b"] = R.bf16(0.1 * w["l0.mix.q.b"])
    w["l0.mix.q"] = _replace(w["l0.mix.q"], h[seeker], 3.0 * want - w["l0.mix.q.b"])
    return cfg, w, beacon, seeker


def seen_matters(cfg, w, prompt, place):
    """How far the last position's logits move with another token at `place`."""
    other = np.array(prompt)
    other[place] = 60
    a, b = R.forward(cfg, w, prompt), R.forward(cfg, w, other)
    return np.sqrt(np.mean((a[-1] - b[-1]) ** 2)) / np.sqrt(np.mean(a ** 2))


@BOTH
@pytest.mark.parametrize("size,keep", [(20, 3), (64, 0), (130, 5), (16, 17), (7, 130)])
def test_window_edges_and_kept_tokens(size, keep, dtype):
    """The marked key just inside and just outside the window, among the kept first tokens and just after them, found by a
    prompt and by a decoded token; portions that end around the edges."""
    cfg, w, beacon, seeker = window_model(size, keep)
    h = Harness(cfg, w, dtype, pool_tokens=2048, step_tokens=1400)
    rng = np.random.default_rng(size)
    filler = lambda n: rng.integers(5, cfg["vocab"], n)
    n_long = 300 + size
    cases = [(n_long - size, True, "window_in"), (n_long - size - 1, False, "window_out")]   # the seeker stands at n_long - 1
    if keep:
        cases += [(keep - 1, True, "last kept"), (0, True, "first kept")]
    cases += [(keep, False, "after the kept")]
    for i, (place, seen, what) in enumerate(cases):
        p = filler(n_long)
        p[place], p[-1] = beacon, seeker
        moved = seen_matters(cfg, w, p, place)
        assert (moved > 3 * TOLS["bfloat16"]) == seen and (seen or moved == 0.0), (what, moved)
        for k, cuts in enumerate(([n_long], [n_long - 1, 1], [n_long - size - 1, size - 1, 2] if size > 1 else [n_long - 2, 2], [place + 1, n_long - place - 1])):
            sid = (i, k)
            h.known(sid, p)
            at = 0
            for c in cuts:
                if c:
                    h.run([(sid, p[at:at + c])])
                    at += c
            h.drop(sid)
    h.close()


@BOTH
def test_windows_pass_over_decoded_tokens(dtype):
    """The marked key is decoded, and the window slides over it one token at a time."""
    size, keep = 18, 2
    cfg, w, beacon, seeker = window_model(size, keep)
    h = Harness(cfg, w, dtype)
    rng = np.random.default_rng(4)
    p = rng.integers(5, cfg["vocab"], 100)
    p[40] = beacon
    p[41:] = seeker
    h.known("a", p)
    h.run([("a", p[:33])])
    for t in range(33, 100):
        h.run([("a", p[t:t + 1])])
    h.close()


def test_the_sink_takes_weight():
    """With scores far below zero the attention returns nearly nothing; without the added one it would return a mean."""
    cfg, w, _, seeker = window_model(40, 0)
    w["l0.mix.q"][:] = 0.0
    w["l0.mix.k"][:] = 0.0
    w["l0.mix.q.b"][:] = 1.0
    w["l0.mix.k.b"][:] = R.bf16(-np.ones(32))
    w["l0.mix.q.norm"][:] = 3.0
    w["l0.mix.k.norm"][:] = 3.0
    h = Harness(cfg, w, "float32")
    p = tokens(np.random.default_rng(1), cfg, 60)
    h.run([("a", p[:50])])
    for t in range(50, 60):
        h.run([("a", p[t:t + 1])])
    h.close()


def recurrence_model():
    """Decays near one, and one token whose key is a hundred times the others': its trace decides the output of all that
    follow."""
    cfg = config(60, 48, [gla(2, 24, 20, 16.0)], eps=1e-6)
    w = R.random_weights(cfg, 8)
    w["l0.mix.a2.b"][:] = 12.0
    w["l0.mix.a2"][:] = R.bf16(0.02 * w["l0.mix.a2"])
    w["embed"][:, 0], w["l0.norm1.b"][0] = 0.0, 0.0
    w["embed"][3, 0] = 3.0
    k = w["l0.mix.k"]
    w["l0.mix.k"] = R.bf16(np.concatenate([8.0 * np.sign(k[:, :1]), 0.04 * k[:, 1:]], axis=1))
    w["l0.norm1b"][:] = R.bf16(4.0 * w["l0.norm1b"])
    return cfg, w


@BOTH
def test_far_tokens_of_the_gated_recurrence(dtype):
    """The state must pass through chunks, cuts and slots, over a thousand tokens and from any place of a chunk."""
    cfg, w = recurrence_model()
    h = Harness(cfg, w, dtype, pool_tokens=2048, step_tokens=1400)
    rng = np.random.default_rng(3)
    prompt = rng.integers(5, 60, 1200)
    prompt[20] = 3
    other = prompt.copy()
    other[20] = 7
    ref = R.forward(cfg, w, prompt)
    assert np.sqrt(np.mean((R.forward(cfg, w, other)[-1] - ref[-1]) ** 2)) > 3 * TOLS["bfloat16"] * np.sqrt(np.mean(ref ** 2))
    for k, cuts in enumerate(([1200], [20, 63, 65, 1, 1, 2, 1048], [1196, 1, 1, 1, 1])):
        h.known(k, prompt)
        at = 0
        for c in cuts:
            h.run([(k, prompt[at:at + c])])
            at += c
        h.drop(k)
    for first in (0, 15, 16, 47, 63, 64, 65, 127):
        p = rng.integers(5, 60, 150)
        p[first] = 3
        h.run([(first, p[:first + 2])])
        h.run([(first, p[first + 2:149])])
        h.run([(first, p[149:])])
        h.drop(first)
    h.close()


def test_a_layer_used_twice_keeps_its_states_apart():
    """Two passes over one layer's tensors differ in their caches and states only."""
    base = [gla(2, 16, 16, 4.0), attention(2, 1, 16, 16, rotation(8), 9, 2, moe(3, 1, 16)), latent(2, 16, rotation(8), 16, 24, 24)]
    cfg = config(70, 48, base + [again(base, 0), again(base, 1), again(base, 2)])
    w = R.random_weights(cfg, 3)
    twice = config(70, 48, base + base)
    w2 = dict(w)
    for k, v in w.items():
        if k[:3] in ("l0.", "l1.", "l2."):
            w2["l%d.%s" % (int(k[1]) + 3, k[3:])] = v
    prompt = tokens(np.random.default_rng(4), cfg, 40)
    zs = []
    for c, ww in ((cfg, w), (twice, w2)):
        h = Harness(c, ww, "float32")
        h.run([("a", prompt[:30])])
        zs.append(np.concatenate([h.run([("a", prompt[t:t + 1])]) for t in range(30, 40)]))
        h.close()
    assert np.array_equal(zs[0], zs[1])


@BOTH
def test_long_decoding_with_reused_pages(dtype):
    cfg = CONFIGS["uneven"]
    h = Harness(cfg, weights("uneven", 21), dtype, pool_tokens=640, max_seqs=2)
    rng = np.random.default_rng(3)
    all_tokens = tokens(rng, cfg, 330)
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
            h.run(rest, check=False) if others else None
            for t in range(25, 30):
                z.append(h.run([("a", a[t:t + 1])] + ([("c", c[:1])] if others else []), check=False)[:1])
            z.append(h.run(([("b", b[:2])] if others else []) + [("a", a[30:])], check=False)[-30:])
            got.append(np.concatenate(z))
            h.close()
        assert np.sqrt(np.mean((got[0] - got[1]) ** 2)) <= tol * np.sqrt(np.mean(got[0] ** 2))


def test_many_sequences_decode_together():
    """Steps of 40 and 140 sequences: every route of the projections, the router and the experts at decode."""
    cfg, w = CONFIGS["uneven"], weights("uneven", 61)
    for n in (40, 140):
        h = Harness(cfg, w, "bfloat16", pool_tokens=16 * n * 2, max_seqs=n, step_tokens=n * 4)
        h.worst = np.inf       # among so many tokens some router nearly ties
        rng = np.random.default_rng(n)
        seqs = [tokens(rng, cfg, 8) for _ in range(n)]
        h.run([(i, s[:4]) for i, s in enumerate(seqs)])
        for t in range(4, 6):
            h.run([(i, s[t:t + 1]) for i, s in enumerate(seqs)])
        h.close()


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
    cfg, w = CONFIGS["narrow"], weights("narrow", 51)    # every expert is chosen: no choice hangs on rounding
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
    r.step([{"id": "b", "tokens": [1] * 128, "want": []}])
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
    empty = {"layers": [{}], **{k: np.zeros(64 * 40, np.uint16) for k in ("embed", "head", "final_norm", "final_norm_b", "final_norm_alpha")}}
    good = attention(2, 1, 8, 8, rotation(4), 8, 2)
    for y in (dict(good, mixer=dict(good["mixer"], dim=300)), dict(good, mixer=dict(good["mixer"], kv_heads=3)), dict(good, mixer=dict(good["mixer"], scale=-1.0)),
              dict(good, mixer=dict(good["mixer"], rot=rotation(3))), dict(good, mlp=moe(600, 2, 8)), dict(good, mlp=moe(2, 3, 8)), dict(good, mlp=moe(64, 40, 8)),
              gla(2, 8, 8, 0.0), gla(2, 300, 8, 1.0), latent(2, 200, rotation(64), 8, 8, 8), latent(2, 8, rotation(8), 8, 8, 1020)):
        with pytest.raises(ComputeError):
            VugedraModel(parse_config(config(64, 40, [y])), empty, 4, 4, 16, 1, 1)


def test_loader_accounts_for_every_tensor(tmp_path):
    cfg, w = CONFIGS["uneven"], weights("uneven", 2)
    for name, change in (("extra", lambda d: d.update(more=np.zeros(3))), ("missing", lambda d: d.pop("l2.mix.a2.b")), ("bias", lambda d: d.pop("l2.norm2b.b")),
                         ("alpha", lambda d: d.pop("l1.norm1.alpha")), ("expert", lambda d: d.pop("l0.mlp.e4.down")),
                         ("shape", lambda d: d.update({"l1.mix.q": d["l1.mix.q"][:-1]})), ("identity", lambda d: d.update({"l0.mlp.router": d["l0.mlp.router"][:-2]}))):
        d = dict(w)
        change(d)
        R.write_checkpoint(tmp_path / name, cfg, d)
        with pytest.raises((ComputeError, IOError)):
            load_model(str(tmp_path / name), Limits(64, 1))
