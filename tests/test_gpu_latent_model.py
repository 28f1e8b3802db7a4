"""The latent-attention decoder through its executor, scheduler and command line against the plain forward pass
of latent_reference.py: a packed step must give every sequence the logits of its whole history run alone,
however the history was cut, batched or placed."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import latent_reference as R
from latent_weights import TINY_LATENT, config, layer, pack
from logismos_b200.cache import BlockAllocator, SlotAllocator
from logismos_b200.embed import ComputeError, InputTooLong
from logismos_b200.generate import generate, sampling_chain
from logismos_b200.latent import LatentModel, parse_config
from logismos_b200.registry import Limits, load_model
from logismos_b200.replay import Replay

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


CONFIGS = {
    # unequal layers: value size above and below the query size, a layer without feed-forward, nothing a multiple of 64
    "uneven": config(301, 136, 3, [layer(5, 24, 40, 72, 80, 200, 1.3), layer(3, 80, 16, 40, 200, 0), layer(2, 130, 70, 50, 144, 90, 0.6)]),
    # many heads, wide latents, one filter tap, a large epsilon
    "heads": config(97, 64, 1, [layer(36, 16, 16, 96, 576, 64, 2.0), layer(18, 64, 64, 64, 320, 128, 0.4)], eps=0.05, cap=3.0),
    # one head of one latent, six taps
    "narrow": config(64, 40, 6, [layer(1, 8, 12, 16, 24, 48, 1.0), layer(2, 12, 8, 8, 16, 0), layer(1, 16, 16, 24, 40, 33, 0.8)], cap=20.0),
    "plain": TINY_LATENT,
}
TOLS = {"float32": 2e-4, "bfloat16": 4e-2}


class Harness:
    def __init__(self, cfg, seed, dtype, pool_tokens=1024, max_seqs=6, step_tokens=700, out_rows=700, block_seed=3):
        self.cfg, self.dtype = cfg, dtype
        self.w = R.random_weights(cfg, seed)
        n = pool_tokens // 16
        self.model = LatentModel(parse_config(cfg), pack(cfg, self.w), n, n, step_tokens, max_seqs, max_seqs, dtype=dtype, max_out_rows=out_rows)
        self.blocks, self.slots, self.hist, self.ref = BlockAllocator(n, n, seed=block_seed), SlotAllocator(max_seqs), {}, {}

    def expect(self, sid):
        """Reference logits of a sequence's whole history (computed once per length)."""
        h = tuple(self.hist[sid])
        if self.ref.get(sid, ((), None))[0] != h:
            self.ref[sid] = (h, R.forward(self.cfg, self.w, h))
        return self.ref[sid][1]

    def run(self, entries, check=True):
        """entries: (sequence, tokens); every new token's logits are compared. Returns greedy tokens of the last rows."""
        ids, cached, new, tabs, sl = [], [], [], [], []
        for sid, toks in entries:
            prev = self.hist.setdefault(sid, [])
            cached.append(len(prev)); new.append(len(toks)); ids.extend(int(t) for t in toks)
            prev.extend(int(t) for t in toks)
            tabs.append(self.blocks.ensure(sid, len(prev))); sl.append(self.slots.get(sid))
        toks = self.model.step(ids, cached, new, np.stack(tabs), sl, out_rows=range(len(ids)))
        assert self.model.device_status() == 0
        z, at = self.model.last_logits(), 0
        assert np.array_equal(toks, z.argmax(1))
        for (sid, t) in entries:
            if check:
                ref = self.expect(sid)
                self.compare(z[at:at + len(t)], ref[len(ref) - len(t):], (sid, len(ref)), ref)
            at += len(t)
        return z

    def compare(self, z, ref, what, scale=None, factor=1.0):
        err = np.sqrt(np.mean((z - ref) ** 2, axis=1)) / np.sqrt(np.mean((ref if scale is None else scale) ** 2))
        assert err.max() <= factor * TOLS[self.dtype], (what, int(err.argmax()), float(err.max()))

    def drop(self, sid):
        self.blocks.release(sid); self.slots.release(sid); self.hist.pop(sid)


def tokens(rng, cfg, n):
    return rng.integers(0, cfg["vocab"], n)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prompt_portions_and_decoding_agree(name, dtype):
    """One token, a whole prompt, the same prompt token by token, and cut into portions down to two tokens, at page
    and tile borders; pages and slots are given back and used again in between."""
    cfg = CONFIGS[name]
    h = Harness(cfg, 11, dtype)
    rng = np.random.default_rng(1)
    h.run([("one", tokens(rng, cfg, 1))])
    prompt = tokens(rng, cfg, 150)
    whole = h.run([("w", prompt)])
    h.drop("one")
    for t in range(40):
        z = h.run([("d", prompt[t:t + 1])])
        h.compare(z, whole[t:t + 1], ("decoded against prompt", t), whole, factor=2.0)   # both sides are rounded
    h.drop("w")
    for k, cuts in enumerate(([2] * 10 + [130], [15, 1, 1, 16, 17, 3, 97], [63, 2, 64, 21], [128, 2, 20], [149, 1])):
        at = 0
        for c in cuts:
            h.run([(k, prompt[at:at + c])])
            at += c
        h.drop(k)
    h.model.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_mixed_batches_of_unequal_requests(name, dtype):
    cfg = CONFIGS[name]
    h = Harness(cfg, 12, dtype)
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
    h.model.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_far_keys_stand_out(dtype):
    """One token's key is scaled up through its embedding and matched by another's query, so that a single far
    score decides the output: it must be found from any distance, across pages, chunks and cuts."""
    cfg = config(120, 64, 2, [layer(2, 32, 32, 64, 64, 0, scale=2.0)])
    h = Harness(cfg, 5, dtype, pool_tokens=2048, step_tokens=1400, out_rows=1400)
    w = h.w
    w["l0.canon1"][:] = 0.0
    beacon, seeker = 3, 4
    # the query of `seeker` is the key of `beacon`: solve W_uk c_beacon = q through the query's own latent
    eps = cfg["norm"]["eps"]
    hh = R.rms_norm(w["embed"], 1.0 + w["l0.norm1"], eps)
    k = R.latent_kv(hh, w["l0.mix.dkv"], w["l0.mix.dkv.norm"], eps) @ w["l0.mix.uk"].T
    cq = R.rms_norm(hh @ w["l0.mix.dq"].T, w["l0.mix.dq.norm"], eps)
    target = k[beacon] / np.linalg.norm(k[beacon]) * 6.0
    a = cq[seeker]
    w["l0.mix.uq"] = R.bf16(w["l0.mix.uq"] * 0.2 + np.outer(target - 0.2 * w["l0.mix.uq"] @ a, a) / (a @ a))
    h.model.close()
    h.model = LatentModel(parse_config(cfg), pack(cfg, w), 128, 128, 1400, 6, 6, dtype=dtype, max_out_rows=1400)
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
    h.run([("d", prompt[:1298])])
    for t in prompt[1298:]:
        h.run([("d", [t])])
    h.drop("d")
    h.run([("c", prompt[:8])])
    h.run([("c", prompt[8:1297])])
    h.run([("c", prompt[1297:1299])])
    for first in (1, 15, 16, 17, 63, 64, 65, 127, 128, 129):    # the beacon just before and after page and tile borders
        p = np.concatenate([filler(first - 1), [beacon], filler(40), [seeker]])
        h.run([(first, p[:-1])])
        h.run([(first, p[-1:])])
        h.drop(first)
    h.model.close()


def test_long_decoding_with_reused_pages():
    cfg = CONFIGS["plain"]
    h = Harness(cfg, 21, "float32", pool_tokens=640, max_seqs=2)
    rng = np.random.default_rng(3)
    all_tokens = tokens(rng, cfg, 330)
    for turn in range(2):                      # the second turn's pages are the first's
        h.run([(turn, all_tokens[:20])])
        out = [h.run([(turn, all_tokens[t:t + 1])], check=False)[0] for t in range(20, 330)]
        h.compare(np.stack(out), h.expect(turn)[20:], turn)
        h.drop(turn)
    h.model.close()


def test_bf16_and_fp32_logits_do_not_depend_on_the_batch():
    """The same tokens alone and among others, with other pages and slots: equal up to rounding."""
    for dtype, tol in (("float32", 1e-5), ("bfloat16", 2e-2)):
        cfg = CONFIGS["uneven"]
        rng = np.random.default_rng(4)
        a, b, c = (tokens(rng, cfg, n) for n in (60, 90, 3))
        got = []
        for block_seed, others in ((1, False), (2, True)):
            h = Harness(cfg, 31, dtype, block_seed=block_seed)
            rest = [("b", b), ("c", c)] if others else []
            z = [h.run(rest[:1] + [("a", a[:25])] + rest[1:], check=False)]
            z = [z[0][len(b) if others else 0:][:25]]
            h.run(rest, check=False) if others else None
            for t in range(25, 30):
                z.append(h.run([("a", a[t:t + 1])] + ([("c", c[:1])] if others else []), check=False)[:1])
            z.append(h.run(([("b", b[:2])] if others else []) + [("a", a[30:])], check=False)[-30:])
            got.append(np.concatenate(z))
            h.model.close()
        assert np.abs(got[0] - got[1]).max() <= tol * np.abs(got[0]).max()


def greedy_reference(cfg, w, prompt, n):
    h = list(prompt)
    margins = []
    for _ in range(n):
        z = R.forward(cfg, w, h)[-1]
        top = np.sort(z)[-2:]
        margins.append(top[1] - top[0])
        h.append(int(z.argmax()))
    return h[len(prompt):], min(margins)


def test_greedy_generation_through_scheduler_and_command_line(tmp_path):
    """Prompts fed in chunks beside decoding sequences, more requests than slots, from a model folder."""
    cfg = CONFIGS["uneven"]
    w = R.random_weights(cfg, 41)
    R.write_checkpoint(tmp_path, cfg, w)
    rng = np.random.default_rng(6)
    prompts = [tokens(rng, cfg, n).tolist() for n in (40, 1, 17, 64, 2)]
    want = [greedy_reference(cfg, w, p, 10) for p in prompts]
    assert min(m for _, m in want) > 1e-4      # no near ties: the continuation is defined
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
    R.write_checkpoint(tmp_path, cfg, R.random_weights(cfg, 42))
    served = load_model(str(tmp_path), Limits(256, 4))
    prompts = [[1, 2, 3], [7], [9, 8]]
    greedy = generate(served, prompts, 8)
    assert generate(served, prompts, 8, sampling_chain(1.0, 1, 1.0, 0.0, 5)) == greedy     # top-1 is greedy
    hot = [generate(served, prompts, 8, sampling_chain(5.0, 0, 1.0, 0.0, s)) for s in (1, 1, 2)]
    assert hot[0] == hot[1] and hot[0] != hot[2] and hot[0] != greedy
    assert all(0 <= t < cfg["vocab"] for p in hot[0] for t in p)
    served.close()


def test_trace_replay_from_a_folder(tmp_path):
    cfg = CONFIGS["plain"]
    w = R.random_weights(cfg, 51)
    R.write_checkpoint(tmp_path / "m", cfg, w)
    rng = np.random.default_rng(8)
    a, b, c = (tokens(rng, cfg, n).tolist() for n in (100, 30, 64))
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:50], "want": [0, 49]}, {"id": "b", "tokens": b[:1], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[1:3], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[3:], "want": [26]}, {"id": "a", "tokens": a[50:51], "want": [0]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "c", "tokens": c, "want": [63, 5]}, {"id": "a", "tokens": a[51:], "want": [48]}], "end": ["a", "c"]}]
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "192"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True)
        assert r.returncode == 0, r.stderr
        assert r.stdout.split("\n")[:4] == ["done 0", "done 1", "done 2", "done 3"]
        assert not (out / "1.f32").exists()
        za, zb, zc = (R.forward(cfg, w, t) for t in (a, b, c))
        for step, ref in ((0, [za[0], za[49]]), (2, [zb[29], za[50]]), (3, [zc[63], zc[5], za[99]])):
            z = np.fromfile(out / f"{step}.f32", "<f4").reshape(len(ref), -1)
            err = np.sqrt(np.mean((z - np.stack(ref)) ** 2, axis=1)) / np.sqrt(np.mean(za ** 2))
            assert err.max() <= TOLS[dtype]


def test_the_cache_pool_and_the_slots_are_finite(tmp_path):
    cfg = CONFIGS["narrow"]
    R.write_checkpoint(tmp_path, cfg, R.random_weights(cfg, 43))
    served = load_model(str(tmp_path), Limits(128, 2))
    r = Replay(served)
    r.step([{"id": "a", "tokens": [1] * 64, "want": []}])
    with pytest.raises(MemoryError):
        r.step([{"id": "b", "tokens": [1] * 65, "want": []}])
    r.end("a"); r.end("b")
    r.step([{"id": "b", "tokens": [1] * 128, "want": []}])
    served.close()


def test_step_rejects_what_it_cannot_run():
    cfg = CONFIGS["narrow"]
    h = Harness(cfg, 1, "bfloat16", pool_tokens=128, max_seqs=2, step_tokens=64, out_rows=4)
    tab = np.arange(8, dtype=np.int32)[None]
    m = h.model
    m.step([1, 2, 3], [0], [3], tab, [0], out_rows=[])
    assert m.last_logits().shape == (0, cfg["vocab"])
    for bad in (lambda: m.step([1], [0], [1], tab, [2]), lambda: m.step([1, 2], [0, 0], [1, 1], np.concatenate([tab, tab]), [1, 1]),
                lambda: m.step([1] * 65, [0], [65], tab, [0]), lambda: m.step([1], [0], [1], tab, [0], out_rows=[1]),
                lambda: m.step([1], [0], [1], tab, [0], out_rows=[0] * 5), lambda: m.step([1], [0], [1], np.full_like(tab, 9), [0])):
        with pytest.raises(ComputeError):
            bad()
    with pytest.raises(InputTooLong):
        m.step([1], [128], [1], tab, [0])
    m.close()
    for y, what in ((layer(1, 300, 8, 8, 8, 0), "head dim"), (layer(1, 8, 8, 8, 2000, 0), "rank"), (layer(1, 8, 8, 8, 8, 0, scale=-1.0), "scale")):
        c = config(64, 40, 2, [y])
        with pytest.raises(ComputeError):
            LatentModel(parse_config(c), pack(c, R.random_weights(c, 1)), 4, 4, 16, 1, 1)


def test_loader_accounts_for_every_tensor(tmp_path):
    cfg = CONFIGS["narrow"]
    w = R.random_weights(cfg, 2)
    for name, change in (("extra", lambda d: d.update(more=np.zeros(3))), ("missing", lambda d: d.pop("l1.dwa")),
                         ("shape", lambda d: d.update({"l0.mix.uq": d["l0.mix.uq"][:-1]}))):
        d = dict(w)
        change(d)
        R.write_checkpoint(tmp_path / name, cfg, d)
        with pytest.raises((ComputeError, IOError)):
            load_model(str(tmp_path / name), Limits(64, 1))
