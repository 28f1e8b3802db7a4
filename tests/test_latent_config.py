"""The latent-attention decoder's host side without a GPU: the oracle's own properties, reading of config.json,
the registry, cache and slot managers, the trace replay over a fake executor, and the partial build."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import latent_reference as R
from logismos_b200 import build, registry
from logismos_b200.cache import BlockAllocator, SlotAllocator, blocks_for
from logismos_b200.generate import generate
from logismos_b200.latent import parse_config
from logismos_b200.registry import Limits, Served
from logismos_b200.replay import Replay

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))

CFG = {"architecture": "Vofosun", "vocab": 50, "width": 24, "canon": {"taps": 3}, "norm": {"eps": 1e-5}, "logit_softcap": 5.0,
       "layers": [{"type": "latent_attention", "mixer": {"heads": 2, "dim": 6, "vdim": 4, "q_rank": 10, "kv_rank": 8, "scale": 0.5},
                   "mlp": {"kind": "dense", "ff": 20, "limit": 0.8}},
                  {"type": "latent_attention", "mixer": {"heads": 3, "dim": 4, "vdim": 7, "q_rank": 6, "kv_rank": 12, "scale": 0.3}, "mlp": None}]}


def test_oracle_is_causal_and_every_mechanism_counts():
    w = R.random_weights(CFG, 3)
    toks = np.random.default_rng(0).integers(0, 50, 12)
    z = R.forward(CFG, w, toks)
    assert np.allclose(R.forward(CFG, w, toks[:7]), z[:7], rtol=0, atol=1e-12)
    other = toks.copy()
    other[3] = (other[3] + 1) % 50
    assert np.abs(R.forward(CFG, w, other) - z)[3:].max(axis=1).min() > 1e-6    # every later position sees token 3
    for name in R.tensor_shapes(CFG):                                           # no tensor is ignored
        d = dict(w)
        d[name] = d[name] * 0.5 + 0.05
        assert np.abs(R.forward(CFG, d, toks) - z).max() > 1e-6, name
    assert np.abs(z).max() <= 5.0


def test_oracle_convolution_by_hand():
    h = np.arange(8.0).reshape(4, 2)
    w = np.array([[1.0, 10.0, 100.0], [0.0, 0.0, 2.0]])
    assert np.array_equal(R.causal_conv(h, w)[:, 0], [0, 200, 20 + 400, 2 * 1 + 40 + 600])
    assert np.array_equal(R.causal_conv(h, w)[:, 1], 2 * h[:, 1])


def test_parse_config():
    c = parse_config(CFG)
    assert (c["vocab"], c["hidden"], c["n_layers"], c["conv_taps"], c["rms_eps"], c["logit_softcap"]) == (50, 24, 2, 3, 1e-5, 5.0)
    assert c["layers"][0] == {"heads": 2, "dim": 6, "vdim": 4, "q_rank": 10, "kv_rank": 8, "scale": 0.5, "ff": 20, "glu_limit": 0.8}
    assert c["layers"][1]["ff"] == 0
    for change in (lambda d: d["layers"][0].update(type="other"), lambda d: d["layers"][0]["mlp"].update(kind="other")):
        d = json.loads(json.dumps(CFG))
        change(d)
        with pytest.raises(ValueError):
            parse_config(d)


def test_registry_picks_by_architecture(tmp_path):
    assert registry.architecture_of(CFG) == "Vofosun"
    assert registry.architecture_of({"architectures": ["Qwen2ForCausalLM"]}) == "Qwen2ForCausalLM"
    for bad in ({}, {"architecture": "nothing"}):
        with pytest.raises(ValueError):
            registry.architecture_of(bad)
    (tmp_path / "config.json").write_text(json.dumps({"architectures": ["Qwen2ForCausalLM"]}))
    with pytest.raises(registry.UnsupportedDtype):
        registry.load_model(str(tmp_path), Limits(64, 1), "float32")
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "64"],
                       input="", capture_output=True, text=True)
    assert r.returncode == 3


def test_allocators_share_nothing_and_take_back():
    b = BlockAllocator(6, 4, seed=None)
    assert blocks_for(0) == 0 and blocks_for(16) == 1 and blocks_for(17) == 2
    r1, r2 = b.ensure("x", 17), b.ensure("y", 33)
    assert sorted(r1[r1 >= 0].tolist() + r2[r2 >= 0].tolist()) == [0, 1, 2, 3, 4] and (r1[2:] == -1).all()
    assert np.array_equal(b.ensure("x", 32), r1) and b.ensure("x", 33)[2] == 5
    with pytest.raises(MemoryError):
        b.ensure("z", 1)
    assert "z" not in b.tables
    with pytest.raises(ValueError):
        b.ensure("x", 65)
    b.release("y"); b.release("nobody")
    assert len(b.free) == 3 and b.ensure("z", 48).max() >= 0
    s = SlotAllocator(2)
    assert {s.get("x"), s.get("y")} == {0, 1} and s.get("x") == s.get("x")
    with pytest.raises(MemoryError):
        s.get("z")
    s.release("x")
    assert s.get("z") in (0, 1)


class FakeModel:
    """An executor whose logits encode the sequence's history; keeps it by state slot and checks what it is given."""

    def __init__(self, vocab):
        self.cfg, self.hist, self.calls = {"vocab": vocab}, {}, []

    def step(self, ids, cached, new, tables, slots, out_rows=None):
        rows, at = [], 0
        assert len(set(slots.tolist())) == len(slots)
        used = [b for t in tables for b in t[t >= 0].tolist()]
        assert len(used) == len(set(used))
        for c, n, t, s in zip(cached, new, tables, slots):
            h = self.hist[s] = ([] if c == 0 else self.hist[s][:c])
            assert len(h) == c and (t[:blocks_for(c + n)] >= 0).all()
            for tok in ids[at:at + n].tolist():
                h.append(tok)
                z = np.zeros(self.cfg["vocab"], np.float32)
                z[(sum(h) * 31 + len(h)) % self.cfg["vocab"]] = 1.0
                rows.append(z)
            at += n
        self.calls.append([int(n) for n in new])
        last = np.cumsum(new) - 1 if out_rows is None else list(out_rows)
        self.logits = np.stack([rows[i] for i in last]) if len(last) else np.zeros((0, self.cfg["vocab"]), np.float32)
        return self.logits.argmax(1).astype(np.uint32)

    def last_logits(self):
        return self.logits


def nxt(h, vocab=50):
    return (sum(h) * 31 + len(h)) % vocab


def test_replay_runs_entries_as_one_batch_and_reuses_what_ended():
    m = FakeModel(50)
    r = Replay(Served("fake", m, True, Limits(128, 2)))
    z = r.step([{"id": "a", "tokens": [1, 2, 3], "want": [2, 0]}, {"id": "b", "tokens": [4], "want": [0]}])
    assert z.argmax(1).tolist() == [nxt([1, 2, 3]), nxt([1]), nxt([4])] and m.calls == [[3, 1]]
    assert r.step([{"id": "a", "tokens": [5], "want": []}]).shape == (0, 50)
    r.end("b")
    z = r.step([{"id": "c", "tokens": [6] * 90, "want": [89]}, {"id": "a", "tokens": [7, 8], "want": [1]}])
    assert z.argmax(1).tolist() == [nxt([6] * 90), nxt([1, 2, 3, 5, 7, 8])]
    assert r.step([]).shape == (0, 50) and len(m.calls) == 3
    r.end("a"); r.end("c")
    assert len(r.blocks.free) == 8 and len(r.slots.free) == 2


def test_generate_feeds_the_scheduler():
    m = FakeModel(50)
    served = Served("fake", m, True, Limits(96, 2, max_step_tokens=20))
    prompts = [[3] * 30, [1], [9, 9]]
    out = generate(served, prompts, 5, prefill_token_budget=16)
    for p, o in zip(prompts, out):
        h = list(p)
        for t in o:
            assert t == nxt(h)
            h.append(t)
    assert len(m.calls) > 6


def test_partial_builds_name_existing_sources():
    for group, names in build.GROUPS.items():
        assert set(names) <= set(build.CU_SOURCES + build.CPP_SOURCES), group
        assert all(os.path.exists(s) for s in build._sources(group))
    assert build.group_library("latent") != build.group_library(None) == build.SO
