"""Configurations of the Zetalorn decoder for tests, and its weights in the executor's layout."""
import numpy as np

import zetalorn_reference as R


def moe(experts, top, ff, count, keep, limit=1.5):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}}


def rotation(dims, base=1000.0, factor=None):
    out = {"dims": dims, "base": base}
    return dict(out, scaling={"factor": factor}) if factor else out


def attention(heads, kv_heads, dim, vdim, size, rot, diff=0.4, mlp=None, scale=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": rot, "scale": scale or 1.3 / np.sqrt(dim), "diff": diff,
                                           "mask": {"size": size}}, "mlp": mlp}


def left(heads, kv_heads, dim, vdim, size, pool, rot, scale=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": rot, "scale": scale or 1.2 / np.sqrt(dim), "mask": {"size": size, "pool": pool}}


def right(dim, vdim, decay):
    return {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}


def parallel(a, b, mlp=None):
    return {"type": "parallel", "mixer": {"left": a, "right": b}, "mlp": mlp}


def config(vocab, width, layers, eps=1e-5, loop=None, logit_scale=0.7):
    out = {"architecture": "Zetalorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers, "logit_scale": logit_scale}
    return dict(out, loop=dict(zip(("start", "stop", "times"), loop))) if loop else out


_A = [parallel(left(6, 2, 20, 28, 24, 5, rotation(12, 80.0)), right(24, 40, (0.5, 0.9, 0.995)), moe(6, 2, 20, 3, 2, 0.8)),
      attention(6, 3, 22, 30, 20, rotation(6, 300.0, 3.0), 0.25, moe(8, 3, 28, 2, 1)),
      parallel(left(3, 3, 30, 22, 9, 4, rotation(30)), right(40, 24, (0.99, 0.2)))]
_B = [attention(4, 1, 64, 128, 70, rotation(64, 5e4), 0.8, moe(12, 1, 40, 4, 1, 7.0)), parallel(left(4, 1, 128, 96, 130, 16, rotation(64, 1e4)), right(128, 64, (0.9, 0.999))),
      attention(2, 2, 40, 48, 200, rotation(40, 1e4, 8.0), 0.1, moe(16, 4, 64, 2, 2, 0.5))]
_C = [parallel(left(20, 1, 8, 8, 5, 1, rotation(2, 50.0)), right(10, 8, (0.7, 1.0, 0.0, 0.95, 0.3)), moe(3, 3, 33, 1, 1)), attention(20, 1, 8, 8, 3, rotation(8, 9.0, 1.5), 0.5),
      parallel(left(1, 1, 16, 9, 33, 40, rotation(10)), right(16, 16, (0.97,)), moe(4, 2, 16, 4, 2))]
_D = [attention(2, 1, 120, 200, 130, rotation(100, 1e4), 0.6, moe(40, 4, 24, 8, 3)), parallel(left(2, 2, 150, 200, 64, 3, rotation(150, 1e4)), right(136, 20, (0.99, 0.4))),
      parallel(left(2, 1, 40, 140, 1, 2, rotation(4)), right(40, 140, (0.98,))), attention(4, 2, 130 - 2, 40, 1, rotation(12), 0.9)]

CONFIGS = {
    # nothing a multiple of 64, grouped keys, a pool that straddles pages, a run of layers repeated three times
    "uneven": config(211, 88, _A, eps=1e-3, loop=(1, 3, 3), logit_scale=1.7),
    # head sizes of real layers, one key head, the first layer repeated with those after it, one expert per token
    "large_heads": config(130, 192, _B, loop=(0, 2, 2)),
    # pools of one token and of more than a page, decays of one and zero, groups of one expert, a large epsilon, no loop
    "narrow": config(64, 40, _C, eps=0.05),
    # heads beyond what the chunk-parallel form takes, more than 32 router outputs, windows and chunks of one token
    "wide_heads": config(97, 72, _D, loop=(3, 4, 2), logit_scale=0.3),
}
TINY_ZETALORN = config(160, 128, [parallel(left(4, 2, 64, 64, 24, 8, rotation(32, 1e4)), right(64, 64, (0.9, 0.99)), moe(8, 2, 64, 2, 1)),
                                  attention(2, 1, 32, 64, 32, rotation(32, 1e4, 4.0), 0.3, moe(8, 2, 64, 4, 2))], loop=(0, 2, 2))


def weights(name, seed):
    return R.random_weights(CONFIGS[name], seed)


def pack(cfg, w):
    b = {k: np.ascontiguousarray(R.bf16_bits(v)) for k, v in w.items()}
    out = {"embed": b["embed"], "head": b["head"], "final_norm": b["final.norm"], "layers": []}
    if cfg.get("loop"):
        out["loop_step"] = b["loop.step"]
    seen = set()
    for i, _ in R.runs(cfg):
        y = {}
        if i not in seen:
            seen.add(i)
            p = "l%d." % i
            for name, v in b.items():
                if not name.startswith(p):
                    continue
                leaf = name[len(p):].removeprefix("mix.").removeprefix("mlp.")
                if not (leaf[0] == "e" and leaf[1].isdigit()):
                    y[leaf.replace(".", "_")] = v
            lc = cfg["layers"][i]
            if lc["mlp"]:
                y["experts"] = [b["%smlp.e%d.%s" % (p, e, n)] for e in range(lc["mlp"]["router"]["experts"]) for n in ("gate", "up", "down")]
        out["layers"].append(y)
    return out
