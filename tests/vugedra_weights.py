"""Configurations of the Vugedra decoder for tests, and its weights in the executor's layout."""
import numpy as np

import vugedra_reference as R


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, identity=0, shared=0):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "identity": identity}}
    return dict(out, shared={"ff": shared}) if shared else out


def rotation(dims, base=1000.0, scaling=None):
    out = {"dims": dims, "base": base}
    if scaling:
        out["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return out


def attention(heads, kv_heads, dim, vdim, rot, size, keep, mlp=None, scale=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": rot, "scale": scale or 1.3 / np.sqrt(dim),
                                           "mask": {"size": size, "keep_first": keep}}, "mlp": mlp}


def gla(heads, dim, vdim, tau, mlp=None):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": mlp}


def latent(heads, dim, rot, vdim, q_rank, kv_rank, mlp=None, scale=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot["dims"], "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "rot": rot,
                                                  "scale": scale or 1.2 / np.sqrt(dim + rot["dims"])}, "mlp": mlp}


def again(layers, i):
    return dict(layers[i], weights_of=i)


def config(vocab, width, layers, eps=1e-5):
    return {"architecture": "Vugedra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


_A = [latent(3, 22, rotation(6, 300.0, (3.0, 40, 8.0, 1.0)), 30, 27, 21, moe(5, 2, 20, identity=2, shared=34)),
      attention(6, 2, 20, 28, rotation(12, 80.0, (2.5, 30, 4.0, 0.7)), 24, 3, dense(50)), gla(3, 24, 40, 4.0, moe(7, 3, 28))]
_B = [attention(4, 1, 128, 96, rotation(64, 5e4, (8.0, 64, 32.0, 1.0)), 70, 0, moe(12, 1, 40, identity=5, shared=40)), gla(2, 128, 64, 16.0),
      latent(20, 96, rotation(32, 1e4), 128, 70, 130, dense(64))]
_C = [gla(5, 10, 8, 1.0, dense(33)), attention(20, 1, 8, 8, rotation(2), 5, 140, moe(3, 3, 16, shared=70)), latent(1, 16, rotation(2, 50.0, (4.0, 16, 2.0, 1.0)), 9, 40, 8)]
_D = [attention(2, 2, 150, 200, rotation(150, 1e4), 130, 129, moe(40, 4, 24, identity=3)), gla(2, 40, 140, 8.0, dense(48)), gla(1, 136, 20, 2.0),
      latent(2, 120, rotation(100, 1e3, (1.5, 200, 16.0, 2.0)), 230, 33, 300)]

CONFIGS = {
    # nothing a multiple of 64, grouped keys, tensors used twice, a shared expert larger than the others
    "uneven": config(211, 88, _A + [again(_A, 1), again(_A, 2), again(_A, 0)], eps=1e-3),
    # head sizes of real layers, one key head, no scaling of the rotation, one expert per token, layers without feed-forward
    "large_heads": config(130, 192, _B + [again(_B, 0)]),
    # many query heads of one key head, more kept tokens than the window holds, every expert chosen, tau 1, a large epsilon
    "narrow": config(64, 40, _C + [again(_C, 1)], eps=0.05),
    # heads beyond what the chunk-parallel form takes, more than 32 router outputs
    "wide_heads": config(97, 72, _D),
}
SIZES = {"uneven": dict(decay_rank=5), "large_heads": dict(decay_rank=40), "narrow": dict(decay_rank=3), "wide_heads": dict(decay_rank=33)}
TINY_VUGEDRA = config(160, 128, [_B[2], attention(4, 2, 64, 64, rotation(32, 1e4, (4.0, 32, 8.0, 1.0)), 20, 2, moe(6, 2, 64, identity=2, shared=64)), _B[1]])


def weights(name, seed):
    return R.random_weights(CONFIGS[name], seed, **SIZES[name])


def pack(cfg, w):
    b = {k: np.ascontiguousarray(R.bf16_bits(v)) for k, v in w.items()}
    out = {"embed": b["embed"], "head": b["head"], "layers": []}
    for n in ("", "_b", "_alpha"):
        out["final_norm" + n] = b["final.norm" + n.replace("_", ".")]
    for i, lc in enumerate(cfg["layers"]):
        p, y = "l%d." % i, {}
        if lc.get("weights_of") is None:
            for name, v in b.items():
                if not name.startswith(p):
                    continue
                leaf = name[len(p):].removeprefix("mix.").removeprefix("mlp.")
                if not (leaf[0] == "e" and leaf[1].isdigit()):
                    y[leaf.replace(".", "_")] = v
            if lc["mlp"] and lc["mlp"]["kind"] == "moe":
                y["experts"] = [b["%smlp.e%d.%s" % (p, e, n)] for e in range(lc["mlp"]["router"]["experts"]) for n in ("gate", "up", "down")]
        out["layers"].append(y)
    return out
