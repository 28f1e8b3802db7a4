"""The Vugedra decoder's host side without a GPU: the oracle's own properties, reading of config.json, the registry and
the partial build."""
import json
import math

import numpy as np
import pytest

import vugedra_reference as R
from logismos_b200 import build, registry
from logismos_b200._lib import lib
from logismos_b200.mixer import ATTENTION, GATED, GLA, LATENT, MIXTURE, TANH_AROUND
from logismos_b200.vugedra import parse_config
from vugedra_weights import CONFIGS, SIZES, again, attention, config, dense, gla, latent, moe, rotation

_BASE = [attention(2, 1, 10, 4, rotation(8, 30.0, (2.0, 200, 4.0, 1.0)), 3, 2, moe(3, 2, 5, identity=1, shared=7)), gla(2, 5, 6, 2.0, dense(9)),
         latent(2, 6, rotation(8, 30.0, (2.0, 200, 4.0, 1.0)), 5, 7, 6, moe(2, 1, 4))]
CFG = config(30, 20, _BASE + [again(_BASE, 0)])


def test_oracle_is_causal_and_every_tensor_counts():
    w = R.random_weights(CFG, 3, decay_rank=3)
    toks = np.random.default_rng(0).integers(0, 30, 14)
    z = R.forward(CFG, w, toks)
    assert np.allclose(R.forward(CFG, w, toks[:8]), z[:8], rtol=0, atol=1e-11)
    other = toks.copy()
    other[3] = (other[3] + 1) % 30
    assert np.abs(R.forward(CFG, w, other) - z)[3:].max(axis=1).min() > 1e-7    # every later position sees token 3
    for name in w:                                                               # no tensor is ignored
        d = dict(w)
        d[name] = d[name] * 0.5 + (1.0 if "correction" in name else 0.05) * np.random.default_rng(1).standard_normal(d[name].shape)
        assert np.abs(R.forward(CFG, d, toks) - z).max() > 1e-6, name
    for layer, path, value in ((0, ("mixer", "scale"), 0.1), (0, ("mixer", "mask", "size"), 5), (0, ("mixer", "mask", "keep_first"), 1), (0, ("mixer", "rot", "base"), 90.0),
                               (0, ("mixer", "rot", "dims"), 6), (0, ("mixer", "rot", "scaling", "factor"), 3.0), (0, ("mixer", "rot", "scaling", "original"), 20),
                               (0, ("mixer", "rot", "scaling", "fast"), 1.5), (0, ("mlp", "router", "top"), 1), (1, ("mixer", "tau"), 3.0), (2, ("mixer", "scale"), 0.1),
                               (2, ("mixer", "rot", "scaling", "slow"), 0.4)):
        c = json.loads(json.dumps(CFG))
        for i in ((0, 3) if layer == 0 else (layer,)):
            at = c["layers"][i]
            for k in path[:-1]:
                at = at[k]
            at[path[-1]] = value
        assert np.abs(R.forward(c, w, toks) - z).max() > 1e-6, path


def test_window_and_kept_tokens_by_hand():
    m = R.window_mask(7, 3, 2)
    assert [list(np.nonzero(r)[0]) for r in m] == [[0], [0, 1], [0, 1, 2], [0, 1, 2, 3], [0, 1, 2, 3, 4], [0, 1, 3, 4, 5], [0, 1, 4, 5, 6]]
    assert [list(np.nonzero(r)[0]) for r in R.window_mask(4, 1, 0)] == [[0], [1], [2], [3]]
    p = R.softmax_plus_one(np.array([[0.0, math.log(2.0), -np.inf]]))
    assert np.allclose(p, [[0.25, 0.5, 0.0]])


def test_rotations():
    rng = np.random.default_rng(2)
    q, k = rng.standard_normal((1, 1, 8)), rng.standard_normal((1, 1, 8))
    rot = rotation(6, 50.0)
    dot = lambda i, j: float((R.rotate(q, [i], rot) * R.rotate(k, [j], rot)).sum())
    assert np.isclose(dot(9, 4), dot(25, 20)) and not np.isclose(dot(9, 4), dot(9, 5))      # distances only
    assert np.array_equal(R.rotate(q, [11], rot)[..., 6:], q[..., 6:])
    # pairs are neighbours: position 1 turns (1, 0) in the first pair by one radian
    assert np.allclose(R.rotate(np.array([[[1.0, 0, 0, 0]]]), [1], rotation(4, 50.0)), [[[math.cos(1), math.sin(1), 0, 0]]])
    # fast pairs keep their frequency, slow ones are divided by the factor, both sides of the ramp
    f, amp = R.rotary_frequencies(rotation(64, 1e4, (8.0, 4096, 32.0, 1.0)))
    plain, one = R.rotary_frequencies(rotation(64, 1e4))
    assert one == 1.0 and np.isclose(amp, 0.1 * math.log(8.0) + 1.0) and f[0] == plain[0] and np.isclose(f[-1], plain[-1] / 8)
    assert ((f <= plain) & (f >= plain / 8 * (1 - 1e-12))).all() and (np.diff(f) < 0).all()


def test_gated_recurrence_carries_its_state():
    rng = np.random.default_rng(1)
    q, k, a = rng.standard_normal((9, 3)), rng.standard_normal((9, 3)), rng.uniform(0, 1, (9, 3))
    v = rng.standard_normal((9, 4))
    o, S = R.gla_recurrence(q, k, v, a)
    o1, S1 = R.gla_recurrence(q[:4], k[:4], v[:4], a[:4])
    o2, S2 = R.gla_recurrence(q[4:], k[4:], v[4:], a[4:], S1)
    assert np.allclose(np.concatenate([o1, o2]), o) and np.allclose(S2, S)
    assert np.allclose(o[0], (q[0] @ k[0]) * v[0])                                          # the first token sees itself
    assert np.allclose(np.exp(R.log_decay(np.array([0.0, 2.0]), 4.0)), (1 / (1 + np.exp(-np.array([0.0, 2.0])))) ** 0.25)


def test_routing_by_hand():
    z = np.log(np.array([[4.0, 2.0, 1.0, 1.0]]))
    e, w = R.route(z, np.zeros(4), 2)
    assert e.tolist() == [[0, 1]] and np.allclose(w, [[2 / 3, 1 / 3]])
    e, w = R.route(z, np.array([0.0, 0.0, 0.0, 0.3]), 2)          # the correction moves the choice, not the weights
    assert e.tolist() == [[0, 3]] and np.allclose(w, [[0.8, 0.2]])


def test_parse_config():
    c = parse_config(CFG)
    assert (c["vocab"], c["hidden"], c["n_layers"], c["norm_eps"], c["norm"]) == (30, 20, 4, 1e-5, TANH_AROUND)
    y = c["layers"][0]
    assert (y["kind"], y["weights_of"], y["heads"], y["kv_heads"], y["dim"], y["vdim"], y["window"], y["keep_first"]) == (ATTENTION, 0, 2, 1, 10, 4, 3, 2)
    assert (y["rot_dims"], y["rot_base"], y["rot_factor"], y["rot_original"], y["rot_fast"], y["rot_slow"]) == (8, 30.0, 2.0, 200.0, 4.0, 1.0)
    assert (y["ff_kind"], y["ff"], y["experts"], y["identity"], y["top"], y["shared_ff"]) == (MIXTURE, 5, 3, 1, 2, 7)
    assert c["layers"][1] == {"kind": GLA, "weights_of": 1, "heads": 2, "dim": 5, "vdim": 6, "tau": 2.0, "ff": 9, "ff_kind": GATED}
    y = c["layers"][2]
    assert (y["kind"], y["q_rank"], y["kv_rank"], y["rot_dims"], y["shared_ff"], y["identity"]) == (LATENT, 7, 6, 8, 0, 0)
    assert c["layers"][3] == c["layers"][0]
    chain = json.loads(json.dumps(CFG))
    chain["layers"].append(dict(chain["layers"][3], weights_of=3))              # of a layer that itself uses another's
    chain["layers"].append(gla(1, 4, 4, 1.0))
    c = parse_config(chain)
    assert c["layers"][4]["weights_of"] == 0 and c["layers"][5]["ff"] == 0


@pytest.mark.parametrize("change", [lambda d: d["layers"][0].update(type="other"), lambda d: d["layers"][0]["mlp"].update(kind="other"),
                                    lambda d: d["layers"][3].update(weights_of=3), lambda d: d["layers"][3].update(weights_of=7),
                                    lambda d: d["layers"][3].update(weights_of=1), lambda d: d["layers"][3]["mixer"].update(scale=2.0),
                                    lambda d: d["layers"][2]["mixer"].update(rot_dim=6), lambda d: d["layers"][1]["mixer"].update(tau="x"),
                                    lambda d: [d["layers"][i]["mixer"]["rot"].update(dims=12) for i in (0, 3)]])
def test_parse_config_rejects(change):
    d = json.loads(json.dumps(CFG))
    change(d)
    with pytest.raises(ValueError):
        parse_config(d)


def test_registry_and_build_group():
    assert registry.architecture_of(CFG) == "Vugedra"
    entry = registry.REGISTRY["Vugedra"]
    assert entry.takes_slots and entry.dtypes == ("bfloat16", "float32")
    assert set(build.GROUPS[entry.build_group]) <= set(build.CU_SOURCES + build.CPP_SOURCES)


def test_keys_that_windows_leave_out():
    """Host arithmetic of the split contexts and of the gather: nothing that a query sees is left out, and what remains
    does not grow with the context."""
    for size, keep in ((1, 0), (5, 3), (16, 16), (17, 15), (128, 0), (130, 129), (40, 300), (0, 0), (1000, 4)):
        for ctx in list(range(1, 60)) + [127, 128, 129, 400, 1000, 5000]:
            v = lib.logismos_window_context(ctx, size, keep)
            gap = ctx - v
            assert gap % 16 == 0 and gap >= 0
            if size == 0:
                assert gap == 0
                continue
            kept = -(-keep // 16) * 16
            assert gap == 0 or kept + gap <= ctx - size              # the first key of the window comes after what is skipped
            assert v <= max(kept + size + 16, min(ctx, kept + size + 16))
            for new in (1, 2, 100):
                if new > ctx:
                    continue
                n = lib.logismos_window_keys(ctx, new, size, keep)
                gap, tiles = ctx - n, -(-keep // 128) * 128
                assert gap % 8 == 0 and (gap == 0 or tiles + gap <= ctx - new - size + 1)
                assert n <= tiles + size + new + 8 or gap == 0


def test_test_configurations_differ_in_everything_that_can():
    layers = [y for c in CONFIGS.values() for y in c["layers"]]
    for kind in ("attention", "gla", "latent_attention"):
        pairs = [(y["mixer"]["dim"], y["mixer"]["vdim"]) for y in layers if y["type"] == kind]
        assert any(a < b for a, b in pairs) and any(a > b for a, b in pairs)
    assert any(y["mlp"] is None for y in layers)
    mixtures = [y["mlp"] for y in layers if y["mlp"] and y["mlp"]["kind"] == "moe"]
    assert any("shared" not in m for m in mixtures) and any(m["shared"]["ff"] > m["expert"]["ff"] for m in mixtures if "shared" in m)
    assert any(not m["router"]["identity"] for m in mixtures) and {m["router"]["top"] for m in mixtures} >= {1, 2, 3}
    masks = [y["mixer"]["mask"] for y in layers if y["type"] == "attention"]
    assert any(m["keep_first"] == 0 for m in masks) and any(m["keep_first"] > m["size"] for m in masks)
    for name, c in CONFIGS.items():
        for shape in R.tensor_shapes(c, **SIZES[name]).values():
            assert all(n >= 1 for n in shape)
