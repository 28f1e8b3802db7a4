"""Configurations of the latent-attention decoder for tests, and its weights in the executor's layout."""
import numpy as np

import latent_reference as R


def layer(heads, dim, vdim, q_rank, kv_rank, ff, limit=1.0, scale=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale or 1.7 / np.sqrt(dim)},
            "mlp": {"kind": "dense", "ff": ff, "limit": limit} if ff else None}


def config(vocab, width, taps, layers, eps=1e-5, cap=6.0):
    return {"architecture": "Vofosun", "vocab": vocab, "width": width, "canon": {"taps": taps}, "norm": {"eps": eps}, "logit_softcap": cap,
            "layers": layers}


TINY_LATENT = config(200, 128, 4, [layer(4, 32, 32, 64, 64, 256, 1.2)] * 2)


def pack(cfg, w):
    b = {k: R.bf16_bits(v) for k, v in w.items()}
    out = {"embed": b["embed"], "final_norm": b["final.norm"], "head": b["head"], "layers": []}
    for i, lc in enumerate(cfg["layers"]):
        p = "l%d." % i
        y = {"norm1": b[p + "norm1"], "conv1": b[p + "canon1"], "dwa": b[p + "dwa"]}
        for n in ("dq", "dq.norm", "uq", "dkv", "dkv.norm", "uk", "uv", "o"):
            y[n.replace(".", "_")] = b[p + "mix." + n]
        if lc["mlp"]:
            y["conv2"] = b[p + "canon2"]
            for n in ("gate", "up", "down"):
                y[n], y[n + "_b"] = b[p + "mlp." + n], b[p + "mlp." + n + ".b"]
        out["layers"].append(y)
    return out
