"""The Katadra decoder's host side without a GPU: the oracle's own properties, reading of config.json, the registry
and the partial build."""
import json
import os

import numpy as np
import pytest

import katadra_reference as R
from katadra_weights import CONFIGS, SIZES, again, config, parallel, ssd
from logismos_b200 import build, registry
from logismos_b200.mixer import PARALLEL, SSD, parse_config

_BASE = [ssd(3, 6, 5, 1, 2, 3, ff=14), parallel(2, 1, 6, 4, 2, 5, ff=11, far=9, every=3)]
CFG = config(30, 20, _BASE + [again(_BASE, 1)])


def test_oracle_is_causal_and_every_tensor_counts():
    w = R.random_weights(CFG, 3, rel_rows=6, decay_rank=3)
    toks = np.random.default_rng(0).integers(0, 30, 14)
    z = R.forward(CFG, w, toks)
    assert np.allclose(R.forward(CFG, w, toks[:8]), z[:8], rtol=0, atol=1e-11)
    other = toks.copy()
    other[3] = (other[3] + 1) % 30
    assert np.abs(R.forward(CFG, w, other) - z)[3:].max(axis=1).min() > 1e-6    # every later position sees token 3
    for name in w:                                                               # no tensor is ignored
        d = dict(w)
        d[name] = d[name] * 0.5 + 0.05
        assert np.abs(R.forward(CFG, d, toks) - z).max() > 1e-6, name
    for path, value in ((("left", "softcap"), 2.0), (("left", "scale"), 0.1), (("left", "bias_max"), 30), (("left_scale",), 0.1), (("right_scale",), 0.1)):
        c = json.loads(json.dumps(CFG))
        for y in c["layers"][1:]:
            m = y["mixer"]
            for k in path[:-1]:
                m = m[k]
            m[path[-1]] = value
        assert np.abs(R.forward(c, w, toks) - z).max() > 1e-6, path
    c = json.loads(json.dumps(CFG))
    for y in c["layers"][1:]:
        y["mixer"]["left"]["q_temp"]["coef"] = 0.0
    assert np.abs(R.forward(c, w, toks) - z)[2:].max() > 1e-6


def test_distance_buckets_by_hand():
    # 8 rows up to 16: one each for 0..3, then 4 for ln(n / 4) / ln 4 in quarters
    got = [R.distance_bucket(n, 8, 16) for n in range(20)]
    assert got == [0, 1, 2, 3, 4, 4, 5, 5, 6, 6, 6, 6, 7, 7, 7, 7, 7, 7, 7, 7]
    assert R.distance_bucket(10 ** 6, 9, 40) == 8 and R.distance_bucket(3, 9, 40) == 3


def test_recurrences_carry_their_state():
    rng = np.random.default_rng(1)
    r, k, w = (rng.uniform(0, 1, (9, 3)) for _ in range(3))
    v, u = rng.standard_normal((9, 4)), rng.standard_normal(3)
    o, S = R.time_mix_recurrence(r, k, v, w, u)
    o1, S1 = R.time_mix_recurrence(r[:4], k[:4], v[:4], w[:4], u)
    o2, S2 = R.time_mix_recurrence(r[4:], k[4:], v[4:], w[4:], u, S1)
    assert np.allclose(np.concatenate([o1, o2]), o) and np.allclose(S2, S)
    assert np.allclose(o[0], (r[0] * u * k[0]).sum() * v[0])                   # the first token sees its bonus only
    x, B, C, dt = rng.standard_normal((9, 4)), rng.standard_normal((9, 3)), rng.standard_normal((9, 3)), rng.uniform(0.1, 1, 9)
    y, S = R.ssd_recurrence(x, B, C, dt, 0.3, 0.7)
    y1, S1 = R.ssd_recurrence(x[:5], B[:5], C[:5], dt[:5], 0.3, 0.7)
    y2, S2 = R.ssd_recurrence(x[5:], B[5:], C[5:], dt[5:], 0.3, 0.7, S1)
    assert np.allclose(np.concatenate([y1, y2]), y) and np.allclose(S2, S)
    assert np.allclose(y[0], dt[0] * (B[0] @ C[0]) * x[0] + 0.7 * x[0])


def test_parse_config():
    c = parse_config(CFG)
    assert (c["vocab"], c["hidden"], c["n_layers"], c["norm_eps"]) == (30, 20, 3, 1e-5)
    assert c["layers"][0] == {"kind": SSD, "weights_of": 0, "ff": 14, "ssd_heads": 3, "ssd_vdim": 6, "ssd_state": 5, "ssd_groups": 1, "ssd_norm_groups": 2, "ssd_taps": 3}
    y = c["layers"][1]
    assert (y["kind"], y["weights_of"], y["heads"], y["kv_heads"], y["dim"], y["vdim"], y["bias_max"], y["temp_every"]) == (PARALLEL, 1, 2, 1, 6, 4, 9, 3.0)
    assert (y["tm_heads"], y["tm_dim"], y["left_scale"], y["right_scale"], y["softcap"]) == (2, 5, 0.8, 1.3, 9.0)
    assert c["layers"][2] == y
    chain = json.loads(json.dumps(CFG))
    chain["layers"].append(dict(chain["layers"][2], weights_of=2))              # of a layer that itself uses another's
    assert parse_config(chain)["layers"][3]["weights_of"] == 1


@pytest.mark.parametrize("change", [lambda d: d["layers"][0].update(type="other"), lambda d: d["layers"][0]["mlp"].update(kind="other"),
                                    lambda d: d["layers"][2].update(weights_of=2), lambda d: d["layers"][2].update(weights_of=7),
                                    lambda d: d["layers"][2].update(weights_of=0), lambda d: d["layers"][2]["mixer"].update(left_scale=2.0)])
def test_parse_config_rejects(change):
    d = json.loads(json.dumps(CFG))
    change(d)
    with pytest.raises(ValueError):
        parse_config(d)


def test_registry_and_build_group():
    assert registry.architecture_of(CFG) == "Katadra"
    entry = registry.REGISTRY["Katadra"]
    assert entry.takes_slots and entry.dtypes == ("bfloat16", "float32")
    assert set(build.GROUPS[entry.build_group]) <= set(build.CU_SOURCES + build.CPP_SOURCES)
    assert "latent_model.cu" not in build.GROUPS["mixer"]


def test_test_configurations_differ_in_everything_that_can():
    pairs = [(y["mixer"]["left"]["dim"], y["mixer"]["left"]["vdim"]) for c in CONFIGS.values() for y in c["layers"] if y["type"] == "parallel"]
    assert any(a < b for a, b in pairs) and any(a > b for a, b in pairs)
    for name, c in CONFIGS.items():
        for shape in R.tensor_shapes(c, **SIZES[name]).values():
            assert min(shape) >= 1
