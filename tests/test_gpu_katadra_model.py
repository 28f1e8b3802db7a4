"""The Katadra decoder through its executor, scheduler and command line against the plain forward pass of
katadra_reference.py: a packed step must give every sequence the logits of its whole history run alone, however the
history was cut, batched or placed."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import katadra_reference as R
import stack_harness
from katadra_weights import CONFIGS, SIZES, again, config, pack, parallel, ssd, weights
from logismos_b200.embed import ComputeError, InputTooLong
from logismos_b200.generate import generate, sampling_chain
from logismos_b200.mixer import MixerModel, parse_config
from logismos_b200.registry import Limits, load_model
from logismos_b200.replay import Replay
from stack_harness import TOLS, greedy_reference, tokens

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def Harness(cfg, w, dtype, **kw):
    return stack_harness.Harness(MixerModel, pack, R.forward, cfg, w, dtype, **kw)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
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


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prompt_portions_and_decoding_agree(name, dtype):
    """One token, a whole prompt, the same prompt token by token, and cut into portions down to two tokens, at page
    and chunk borders; pages and slots are given back and used again in between."""
    cfg = CONFIGS[name]
    h = Harness(cfg, weights(name, 11), dtype)
    rng = np.random.default_rng(1)
    h.run([("one", tokens(rng, cfg, 1))])
    prompt = tokens(rng, cfg, 150)
    whole = h.run([("w", prompt)])
    h.drop("one")
    for t in range(40):
        z = h.run([("d", prompt[t:t + 1])], check=False)
        h.compare(z, whole[t:t + 1], ("decoded against prompt", t), whole, factor=2.0)   # both sides are rounded
    h.drop("w")
    for k, cuts in enumerate(([2] * 10 + [130], [15, 1, 1, 16, 17, 3, 97], [63, 2, 64, 21], [128, 2, 20], [149, 1], [1, 2, 3, 144])):
        at = 0
        h.known(k, prompt)
        for c in cuts:
            h.run([(k, prompt[at:at + c])])
            at += c
        h.drop(k)
    h.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
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


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_far_keys_stand_out(dtype):
    """One token's key is matched by another's query, so that a single far score decides the output: it must be found
    from any distance, across pages, chunks and cuts."""
    cfg = config(120, 64, [parallel(2, 1, 32, 32, 1, 16, far=40, coef=0.0, cap=40.0, scale=0.6, left=3.0, right=0.1)], eps=1e-6)
    w = R.random_weights(cfg, 5)
    beacon, seeker = 3, 4
    hh = w["embed"]
    k = R.unit_rms(hh @ w["l0.mix.left.k"].T, 1e-6)
    for a in range(2):   # the query of `seeker` is the key of `beacon`
        q = w["l0.mix.left.q"][32 * a:32 * a + 32]
        w["l0.mix.left.q"][32 * a:32 * a + 32] = R.bf16(0.3 * q + np.outer(3.0 * k[beacon] - 0.3 * q @ hh[seeker], hh[seeker]) / (hh[seeker] @ hh[seeker]))
    w["l0.mix.left.rel"][:] = R.bf16(0.3 * w["l0.mix.left.rel"])
    h = Harness(cfg, w, dtype, pool_tokens=2048, step_tokens=1400)
    rng = np.random.default_rng(9)
    filler = lambda n: rng.integers(5, cfg["vocab"], n)
    prompt = np.concatenate([filler(7), [beacon], filler(1290), [seeker], filler(3)])
    ref = R.forward(cfg, w, prompt)
    without = prompt.copy()
    without[7] = 60
    moved = np.sqrt(np.mean((ref[-4] - R.forward(cfg, w, without)[-4]) ** 2)) / np.sqrt(np.mean(ref ** 2))
    assert moved > 3 * TOLS["bfloat16"]      # the far key decides this position
    h.run([("w", prompt)])
    h.drop("w")
    for sid, cuts in (("d", [1298, 1, 1, 1, 1]), ("c", [8, 1289, 2])):
        at = 0
        h.known(sid, prompt)
        for c in cuts:
            h.run([(sid, prompt[at:at + c])])
            at += c
        h.drop(sid)
    for first in (1, 15, 16, 17, 39, 40, 41, 63, 64, 65, 127, 128, 129):    # the beacon around page, table and tile borders
        p = np.concatenate([filler(first - 1), [beacon], filler(40), [seeker]])
        h.run([(first, p[:-1])])
        h.run([(first, p[-1:])])
        h.drop(first)
    h.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_every_distance_in_prompts_and_decoding(dtype):
    """A steep bias by distance: a bucket border that is one token off changes the output."""
    cfg = config(90, 64, [parallel(2, 2, 16, 24, 1, 8, far=26, coef=0.0, left=2.0, right=0.1)])
    w = R.random_weights(cfg, 6, rel_rows=8)
    w["l0.mix.left.rel"][:] = R.bf16(5.0 * np.random.default_rng(1).standard_normal((8, 2)))
    h = Harness(cfg, w, dtype)
    prompt = tokens(np.random.default_rng(2), cfg, 90)
    h.known("p", prompt)
    h.run([("p", prompt)])
    h.drop("p")
    h.known("d", prompt)
    h.run([("d", prompt[:20])])
    for t in range(20, 90):
        h.run([("d", prompt[t:t + 1])])
    h.close()


def test_a_layer_used_twice_keeps_its_states_apart():
    """Two passes over one layer's tensors differ in their caches and states only."""
    base = [ssd(2, 16, 16, 1, 1, 3), parallel(2, 1, 16, 16, 2, 16)]
    cfg = config(70, 48, base + [again(base, 0), again(base, 1)])
    w = R.random_weights(cfg, 3)
    twice = config(70, 48, base + base)
    w2 = dict(w)
    for k, v in w.items():
        if k[:3] in ("l0.", "l1."):
            w2["l%d.%s" % (int(k[1]) + 2, k[3:])] = v
    prompt = tokens(np.random.default_rng(4), cfg, 40)
    zs = []
    for c, ww in ((cfg, w), (twice, w2)):
        h = Harness(c, ww, "float32")
        h.run([("a", prompt[:30])])
        zs.append(np.concatenate([h.run([("a", prompt[t:t + 1])]) for t in range(30, 40)]))
        h.close()
    assert np.array_equal(zs[0], zs[1])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
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
    good = parallel(2, 1, 8, 8, 1, 8)
    for change in (lambda y: y["mixer"]["left"].update(dim=300), lambda y: y["mixer"]["left"].update(kv_heads=3), lambda y: y["mixer"]["left"].update(scale=-1.0),
                   lambda y: y["mixer"]["left"].update(bias_max=4), lambda y: y["mixer"]["right"].update(dim=300)):
        y = json.loads(json.dumps(good))
        w = R.random_weights(config(64, 40, [y]), 1)
        change(y)
        with pytest.raises(ComputeError):
            MixerModel(parse_config(config(64, 40, [y])), pack(config(64, 40, [good]), w), 4, 4, 16, 1, 1)
    for y in (ssd(3, 8, 8, 2, 1, 2), ssd(2, 8, 8, 1, 3, 2), ssd(2, 8, 8, 1, 1, 9), ssd(2, 300, 8, 1, 1, 2)):
        with pytest.raises(ComputeError):
            MixerModel(parse_config(config(64, 40, [y])), {"layers": [{}], **{k: np.zeros(64 * 40, np.uint16) for k in ("embed", "head", "final_norm", "final_norm_b")}}, 4, 4, 16, 1, 1)


def test_loader_accounts_for_every_tensor(tmp_path):
    cfg, w = CONFIGS["uneven"], weights("uneven", 2)
    for name, change in (("extra", lambda d: d.update(more=np.zeros(3))), ("missing", lambda d: d.pop("l0.mix.right.u")), ("bias", lambda d: d.pop("l2.norm2.b")),
                         ("shape", lambda d: d.update({"l1.mix.in": d["l1.mix.in"][:-1]})), ("table", lambda d: d.update({"l0.mix.left.rel": d["l0.mix.left.rel"][:1]}))):
        d = dict(w)
        change(d)
        R.write_checkpoint(tmp_path / name, cfg, d)
        with pytest.raises((ComputeError, IOError)):
            load_model(str(tmp_path / name), Limits(64, 1))
