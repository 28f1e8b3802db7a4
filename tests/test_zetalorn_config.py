"""The Zetalorn decoder's host side without a GPU: the oracle's own properties, reading of config.json, the registry and the
partial build, and the arithmetic of windows, chunks and pooled blocks."""
import ctypes as C
import json
import math

import numpy as np
import pytest

import zetalorn_reference as R
from logismos_b200 import build, registry
from logismos_b200._lib import lib
from logismos_b200.mixer import DIFF, MIXTURE, PAIR, RMS_GATED, SIGMOID
from logismos_b200.structs import Window
from logismos_b200.zetalorn import parse_config, runs
from zetalorn_weights import CONFIGS, attention, config, left, moe, parallel, right, rotation

CFG = config(30, 20, [parallel(left(2, 1, 10, 4, 3, 2, rotation(8, 30.0)), right(5, 6, (0.8, 0.6)), moe(4, 2, 5, 2, 1, 0.5)),
                      attention(4, 2, 6, 5, 5, rotation(4, 30.0, 2.0), 0.3, moe(3, 2, 4, 1, 1, 0.7)), attention(1, 1, 4, 4, 7, rotation(4), 0.6)], loop=(0, 2, 2))


def test_oracle_is_causal_and_everything_counts():
    w = R.random_weights(CFG, 3)
    toks = np.random.default_rng(0).integers(0, 30, 14)
    z = R.forward(CFG, w, toks)
    assert np.allclose(R.forward(CFG, w, toks[:8]), z[:8], rtol=0, atol=1e-11)
    other = toks.copy()
    other[3] = (other[3] + 1) % 30
    assert np.abs(R.forward(CFG, w, other) - z)[3:].max(axis=1).min() > 1e-9    # every later position sees token 3
    for name in w:                                                               # no tensor is ignored
        d = dict(w)
        d[name] = d[name] * 0.5 + 0.05 * np.random.default_rng(1).standard_normal(d[name].shape)
        assert np.abs(R.forward(CFG, d, toks) - z).max() > 1e-7, name
    for path, value in ((("layers", 0, "mixer", "left", "scale"), 0.1), (("layers", 0, "mixer", "left", "mask", "size"), 4), (("layers", 0, "mixer", "left", "mask", "pool"), 3),
                        (("layers", 0, "mixer", "left", "rot", "base"), 90.0), (("layers", 0, "mixer", "left", "rot", "dims"), 6), (("layers", 0, "mixer", "right", "decay", 1), 0.5),
                        (("layers", 0, "mlp", "expert", "limit"), 0.4), (("layers", 0, "mlp", "router", "top"), 1), (("layers", 0, "mlp", "router", "groups", "keep"), 2),
                        (("layers", 1, "mixer", "mask", "size"), 6), (("layers", 1, "mixer", "diff"), 0.2), (("layers", 1, "mixer", "scale"), 0.2),
                        (("layers", 1, "mixer", "rot", "scaling", "factor"), 3.0), (("layers", 1, "mixer", "rot", "dims"), 2), (("norm", "eps"), 1e-2), (("logit_scale",), 0.5),
                        (("loop", "start"), 1), (("loop", "stop"), 1)):
        c = json.loads(json.dumps(CFG))
        at = c
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        assert np.abs(R.forward(c, w, toks) - z).max() > 1e-7, path


def test_masks_by_hand():
    assert [list(np.nonzero(r)[0]) for r in R.chunk_mask(5, 2)] == [[0], [0, 1], [2], [2, 3], [4]]
    assert [list(np.nonzero(r)[0]) for r in R.window_mask(4, 2)] == [[0], [0, 1], [1, 2], [2, 3]]
    # blocks (0, 1), (2, 3), (4, 5): position 3 sees the first one through a window of two, position 4 has lost token 2 and not yet its block
    assert [list(np.nonzero(r)[0]) for r in R.pooled_mask(7, 2, 2)] == [[], [], [], [0], [0], [0, 1], [0, 1]]
    x = np.arange(10.0).reshape(5, 1, 2)
    assert np.array_equal(R.pooled(x, 2), [[[1, 2]], [[5, 6]]])


def test_pooled_blocks_of_equal_keys_stand_for_one_key():
    """With all keys equal the softmax counts tokens of the window and blocks alike."""
    rng = np.random.default_rng(1)
    v = rng.standard_normal((12, 1, 3))
    o = R.pooled_window_attention(np.ones((12, 1, 2)), np.ones((12, 1, 2)), v, 0.7, 4, 3)
    assert np.allclose(o[11, 0], np.concatenate([v[8:12, 0], R.pooled(v, 3)[:2, 0]]).mean(axis=0))
    assert np.allclose(o[5, 0], v[2:6, 0].mean(axis=0))


def test_rotations():
    rng = np.random.default_rng(2)
    q, k = rng.standard_normal((1, 1, 8)), rng.standard_normal((1, 1, 8))
    rot = rotation(6, 50.0)
    for halves in (False, True):
        dot = lambda i, j: float((R.rotate(q, [i], rot, halves) * R.rotate(k, [j], rot, halves)).sum())
        assert np.isclose(dot(9, 4), dot(25, 20)) and not np.isclose(dot(9, 4), dot(9, 5))      # distances only
        assert np.array_equal(R.rotate(q, [11], rot, halves)[..., 6:], q[..., 6:])
    one = np.array([[[1.0, 0, 0, 0]]])
    assert np.allclose(R.rotate(one, [1], rotation(4, 50.0), False), [[[math.cos(1), math.sin(1), 0, 0]]])
    assert np.allclose(R.rotate(one, [1], rotation(4, 50.0), True), [[[math.cos(1), 0, math.sin(1), 0]]])
    assert np.allclose(R.rotary_frequencies(rotation(8, 50.0, 4.0)), R.rotary_frequencies(rotation(8, 50.0)) / 4)


def test_difference_and_recurrence_by_hand():
    a1, a2 = np.array([[[3.0, 1.0]]]), np.array([[[1.0, 1.0]]])
    assert np.allclose(R.difference(a1, a2, 1.0, 0.25, 0.0), [[[math.sqrt(2) * 0.75, 0.0]]])
    one = {"lq1": np.array([2.0, 0]), "lk1": np.array([0.5, 9]), "lq2": np.zeros(2), "lk2": np.ones(2)}
    assert np.isclose(R.difference_weight(one, 0.3), math.e - 1 + 0.3)
    rng = np.random.default_rng(1)
    q, k, v = rng.standard_normal((9, 3)), rng.standard_normal((9, 3)), rng.standard_normal((9, 4))
    o, S = R.decay_recurrence(q, k, v, 0.7)
    o1, S1 = R.decay_recurrence(q[:4], k[:4], v[:4], 0.7)
    o2, S2 = R.decay_recurrence(q[4:], k[4:], v[4:], 0.7, S1)
    assert np.allclose(np.concatenate([o1, o2]), o) and np.allclose(S2, S)
    assert np.allclose(o[1], (q[1] @ k[1]) * v[1] + 0.7 * (q[1] @ k[0]) * v[0])


def test_routing_by_hand():
    logit = lambda s: np.log(np.array(s) / (1 - np.array(s)))
    z = logit([[0.9, 0.1, 0.1, 0.6, 0.55, 0.5]])
    e, w = R.route(z, 2, 2, 1)                      # the second group's two best outweigh the first's
    assert e.tolist() == [[3, 4]] and np.allclose(w, [[0.6 / 1.15, 0.55 / 1.15]])
    e, w = R.route(z, 2, 2, 2)
    assert e.tolist() == [[0, 3]] and np.allclose(w, [[0.6, 0.4]])
    e, _ = R.route(z, 2, 6, 2)                      # groups of one
    assert e.tolist() == [[0, 3]]


def test_clamped_units_by_hand():
    w = {"gate": np.array([[1.0]]), "up": np.array([[1.0]]), "down": np.array([[1.0]])}
    y = R.clamped_unit(np.array([[9.0], [-9.0], [0.5]]), w, 2.0)[:, 0]
    s = lambda x: 1 / (1 + math.exp(-1.702 * x))
    assert np.allclose(y, [2 * s(2) * 3, -9 * s(-9) * -1, 0.5 * s(0.5) * 1.5])


def test_runs_of_a_loop():
    assert runs(3, None) == [(0, None), (1, None), (2, None)]
    assert runs(4, {"start": 1, "stop": 3, "times": 2}) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    assert runs(2, {"start": 0, "stop": 1, "times": 1}) == [(0, 0), (1, None)]
    for name, c in CONFIGS.items():
        assert runs(len(c["layers"]), c.get("loop")) == R.runs(c), name


def test_parse_config():
    c = parse_config(CFG)
    assert (c["vocab"], c["hidden"], c["n_layers"], c["norm_eps"], c["norm"], c["passes"], c["logit_scale"]) == (30, 20, 5, 1e-5, RMS_GATED, 2, 0.7)
    y = c["layers"][0]
    assert (y["kind"], y["weights_of"], y["file_layer"], y["pass"], y["heads"], y["kv_heads"], y["dim"], y["vdim"], y["window"], y["pool"]) == (PAIR, 0, 1, 1, 2, 1, 10, 4, 3, 2)
    assert (y["rot_dims"], y["rot_base"], y["rot_halves"], y["lin_heads"], y["lin_dim"], y["lin_vdim"], y["decay"]) == (8, 30.0, 1, 2, 5, 6, [0.8, 0.6]) and "rot_factor" not in y
    assert (y["ff_kind"], y["ff"], y["experts"], y["top"], y["scoring"], y["route_groups"], y["keep_groups"], y["glu_limit"], y["no_correction"]) == (MIXTURE, 5, 4, 2, SIGMOID, 2, 1, 0.5, 1)
    y = c["layers"][1]
    assert (y["kind"], y["chunked"], y["window"], y["diff"], y["rot_halves"], y["rot_factor"], y["pass"]) == (DIFF, 1, 5, 0.3, 0, 2.0, 0)
    assert c["layers"][2] == {**c["layers"][0], "pass": 2} and c["layers"][3] == c["layers"][1]
    assert (c["layers"][4]["weights_of"], c["layers"][4]["file_layer"], c["layers"][4]["ff"]) == (4, 3, 0)
    plain = json.loads(json.dumps(CFG))
    del plain["loop"]
    assert parse_config(plain)["passes"] == 0 and [y["pass"] for y in parse_config(plain)["layers"]] == [0, 0, 0]


@pytest.mark.parametrize("change", [lambda d: d["layers"][0].update(type="other"), lambda d: d["layers"][0]["mlp"].update(kind="other"), lambda d: d["loop"].update(stop=4),
                                    lambda d: d["loop"].update(times=0), lambda d: d["loop"].update(start=2), lambda d: d["layers"][0]["mixer"]["right"].update(heads=3),
                                    lambda d: d["layers"][1]["mixer"]["rot"].update(dims=12), lambda d: d["layers"][1]["mixer"].update(diff="x"),
                                    lambda d: d["layers"][0]["mlp"]["expert"].update(limit=0.0)])
def test_parse_config_rejects(change):
    d = json.loads(json.dumps(CFG))
    change(d)
    with pytest.raises(ValueError):
        parse_config(d)


def test_registry_and_build_group():
    assert registry.architecture_of(CFG) == "Zetalorn"
    entry = registry.REGISTRY["Zetalorn"]
    assert entry.takes_slots and entry.dtypes == ("bfloat16", "float32")
    assert {"mixer_paired.cu", "gated_residual.cu"} <= set(build.GROUPS[entry.build_group]) <= set(build.CU_SOURCES + build.CPP_SOURCES)


def test_split_contexts_and_gathers():
    """Host arithmetic: the leading blocks or rows and the window's keys, and nothing besides what rounding takes along."""
    up = lambda v, m: -(-v // m) * m
    for size, pool, chunked in ((1, 1, 0), (5, 3, 0), (16, 16, 0), (40, 8, 0), (130, 5, 0), (9, 40, 0), (1, 0, 1), (7, 0, 1), (64, 0, 1), (130, 0, 1), (33, 0, 0)):
        w = Window(scale=1.0, size=size, chunked=chunked, pool=pool)
        first = lambda i: i - i % size if chunked else max(0, i - size + 1)
        means = lambda i: max(0, i - size + 1) // pool if pool else 0
        for ctx in list(range(1, 70)) + [127, 128, 129, 400, 1000, 5000]:
            i = ctx - 1
            v = lib.logismos_window_view_context(C.byref(w), ctx)
            assert v == up(means(i), 16) + ctx - first(i) // 16 * 16, (size, pool, ctx)
            for new in (1, 2, 100):
                if new <= ctx:
                    n = lib.logismos_window_view_keys(C.byref(w), ctx, new)
                    assert n == up(means(i), 128) + ctx - first(ctx - new) // 8 * 8, (size, pool, ctx, new)


def test_test_configurations_differ_in_everything_that_can():
    layers = [y for c in CONFIGS.values() for y in c["layers"]]
    attn = [y["mixer"] for y in layers if y["type"] == "attention"]
    pairs = [y["mixer"] for y in layers if y["type"] == "parallel"]
    for ms in (attn, [m["left"] for m in pairs], [m["right"] for m in pairs]):
        assert any(m["dim"] < m["vdim"] for m in ms) and any(m["dim"] > m["vdim"] for m in ms)
    for ms in (attn, [m["left"] for m in pairs]):
        assert any(m["kv_heads"] == 1 < m["heads"] for m in ms) and any(m["kv_heads"] == m["heads"] for m in ms) and any(1 < m["kv_heads"] < m["heads"] for m in ms)
        assert any(m["rot"]["dims"] == m["dim"] for m in ms) and any(m["rot"]["dims"] < m["dim"] for m in ms)
    assert any("scaling" in m["rot"] for m in attn) and any("scaling" not in m["rot"] for m in attn)
    masks = [m["left"]["mask"] for m in pairs]
    assert {m["pool"] for m in masks} >= {1, 2, 3, 16, 40} and any(m["size"] < m["pool"] for m in masks) and any(m["size"] % m["pool"] for m in masks)
    assert {m["mask"]["size"] for m in attn} >= {1, 3, 20}
    decays = [d for m in pairs for d in m["right"]["decay"]]
    assert 0.0 in decays and 1.0 in decays
    routers = [y["mlp"]["router"] for y in layers if y["mlp"]]
    assert any(y["mlp"] is None for y in layers) and {r["top"] for r in routers} >= {1, 2, 3, 4}
    assert any(r["groups"]["count"] == 1 for r in routers) and any(r["groups"]["keep"] == r["groups"]["count"] for r in routers) and any(r["groups"]["keep"] == 1 < r["groups"]["count"] for r in routers)
    assert len({y["mlp"]["expert"]["limit"] for y in layers if y["mlp"]}) >= 4
    loops = [c.get("loop") for c in CONFIGS.values()]
    assert None in loops and any(lp and lp["start"] == 0 for lp in loops) and any(lp and lp["times"] == 3 for lp in loops)
