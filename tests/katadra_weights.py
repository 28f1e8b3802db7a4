"""Configurations of the Katadra decoder for tests, and its weights in the executor's layout."""
import numpy as np

import katadra_reference as R


def ssd(heads, vdim, state, groups, norm_groups, taps, ff=0):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": taps},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def parallel(heads, kv_heads, dim, vdim, tm_heads, tm_dim, ff=0, far=60, coef=0.4, every=24, cap=9.0, scale=None, left=0.8, right=1.3):
    return {"type": "parallel", "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "bias_max": far, "scale": scale or 1.5 / np.sqrt(dim),
                                                   "softcap": cap, "q_temp": {"coef": coef, "every": every}},
                                          "right": {"heads": tm_heads, "dim": tm_dim}, "left_scale": left, "right_scale": right},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def again(layers, i):
    return dict(layers[i], weights_of=i)


def config(vocab, width, layers, eps=1e-5):
    return {"architecture": "Katadra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


_A = [parallel(6, 2, 24, 40, 3, 24, 72), ssd(5, 12, 20, 1, 2, 3), ssd(4, 16, 32, 2, 1, 5, ff=60)]
_B = [ssd(8, 64, 128, 2, 8, 4), parallel(4, 1, 128, 96, 2, 64, 0, far=17, every=7.0, left=1.4, right=0.5), ssd(2, 128, 64, 2, 2, 2, ff=128)]
_C = [ssd(6, 8, 10, 3, 2, 1), ssd(1, 40, 16, 1, 5, 8), parallel(20, 1, 8, 8, 1, 100, 33, far=300, cap=30.0, coef=0.0)]
_D = [parallel(2, 2, 150, 200, 1, 130, 64), ssd(2, 140, 136, 1, 7, 4)]

CONFIGS = {
    # nothing a multiple of 64, grouped keys, parts of the norm that cut heads, tensors used twice
    "uneven": config(211, 88, _A + [again(_A, 0), again(_A, 1)], eps=1e-3),
    # head sizes of real layers, one key head
    "large_heads": config(130, 192, _B + [again(_B, 1)]),
    # many query heads of one key head, one and eight taps, a wide bias table, no query temperature, a large epsilon
    "narrow": config(64, 40, _C + [again(_C, 2)], eps=0.05),
    # heads beyond what the chunk-parallel forms take
    "wide_heads": config(97, 72, _D),
}
SIZES = {"uneven": dict(rel_rows=10, decay_rank=5), "large_heads": dict(rel_rows=7, decay_rank=40), "narrow": dict(rel_rows=32, decay_rank=3),
         "wide_heads": dict(rel_rows=12, decay_rank=33)}
TINY_KATADRA = config(160, 128, _B[:2] + [again(_B, 0)])


def weights(name, seed):
    return R.random_weights(CONFIGS[name], seed, **SIZES[name])


def pack(cfg, w):
    b = {k: R.bf16_bits(v) for k, v in w.items()}
    out = {"embed": b["embed"], "final_norm": b["final.norm"], "final_norm_b": b["final.norm.b"], "head": b["head"], "layers": []}
    for i, lc in enumerate(cfg["layers"]):
        p, y = "l%d." % i, {}
        if "weights_of" not in lc:
            for n in ("norm1", "norm2"):
                if p + n in b:
                    y[n], y[n + "_b"] = b[p + n], b[p + n + ".b"]
            for name, v in b.items():
                for part in ("mlp.", "mix."):
                    if name.startswith(p + part) and ".mu." not in name:
                        y[name[len(p + part):].replace(".", "_")] = v
            if lc["type"] == "parallel":
                y["mu"] = [b[p + "mix.right.mu." + s] for s in "rkvgw"]
        out["layers"].append(y)
    return out
