"""Configuration of the Vugedra decoder over the stack-of-mixers executor (``mixer``): tanh norms around every sublayer,
windowed attention with kept first keys and a softmax denominator with one added, gated linear attention, latent attention
with a rotated part; gated feed-forwards, dense or a mixture of experts with identity experts and a shared one."""
from __future__ import annotations

from .mixer import ATTENTION, GATED, GLA, LATENT, MIXTURE, TANH_AROUND, MixerModel, check_shared, weights_owner

KINDS = {"attention": ATTENTION, "gla": GLA, "latent_attention": LATENT}


def _rotation(m: dict, rotated: int) -> dict:
    rot = m.get("rot")
    if not rot:
        return {"rot_dims": 0}
    out = {"rot_dims": int(rot["dims"]), "rot_base": float(rot["base"])}
    if not 0 <= out["rot_dims"] <= rotated:
        raise ValueError(f"{out['rot_dims']} rotated dimensions of {rotated}")
    y = rot.get("scaling")
    if y:
        out.update(rot_factor=float(y["factor"]), rot_original=float(y["original"]), rot_fast=float(y["fast"]), rot_slow=float(y["slow"]))
    return out


def _attention(m: dict) -> dict:
    mask = m.get("mask") or {"size": 0, "keep_first": 0}
    return {"kv_heads": int(m["kv_heads"]), "scale": float(m["scale"]), "window": int(mask["size"]), "keep_first": int(mask.get("keep_first") or 0),
            **_rotation(m, int(m["dim"]))}


def _latent(m: dict) -> dict:
    out = {"q_rank": int(m["q_rank"]), "kv_rank": int(m["kv_rank"]), "scale": float(m["scale"]), **_rotation(m, int(m["rot_dim"]))}
    if out["rot_dims"] != int(m["rot_dim"]):
        raise ValueError("the whole rotated part of a latent head is rotated")
    return out


_MIXERS = {ATTENTION: _attention, GLA: lambda m: {"tau": float(m["tau"])}, LATENT: _latent}


def _feed_forward(mlp) -> dict:
    if not mlp:
        return {"ff": 0}
    if mlp["kind"] == "dense":
        return {"ff": int(mlp["ff"]), "ff_kind": GATED}
    if mlp["kind"] != "moe":
        raise ValueError(f"no feed-forward of kind {mlp['kind']!r}")
    r, shared = mlp["router"], mlp.get("shared")
    return {"ff": int(mlp["expert"]["ff"]), "ff_kind": MIXTURE, "experts": int(r["experts"]), "identity": int(r.get("identity") or 0), "top": int(r["top"]),
            "shared_ff": int(shared["ff"]) if shared else 0}


def parse_config(config: dict) -> dict:
    """config.json of a Vugedra model -> the executor's configuration; the rank of the decays (``tm_rank``) is the
    tensors' own. Raises ValueError for what the design does not have."""
    layers = []
    for i, lc in enumerate(config["layers"]):
        if lc["type"] not in KINDS:
            raise ValueError(f"layer {i}: no mixer of type {lc['type']!r}")
        kind, m = KINDS[lc["type"]], lc["mixer"]
        try:
            layers.append({"kind": kind, "weights_of": weights_owner(config["layers"], i), "heads": int(m["heads"]), "dim": int(m["dim"]), "vdim": int(m["vdim"]),
                           **_MIXERS[kind](m), **_feed_forward(lc.get("mlp"))})
        except ValueError as e:
            raise ValueError(f"layer {i}: {e}") from None
    check_shared(layers)
    return {"vocab": int(config["vocab"]), "hidden": int(config["width"]), "n_layers": len(layers), "norm_eps": float(config["norm"]["eps"]), "norm": TANH_AROUND,
            "layers": layers}


class VugedraModel(MixerModel):
    parse = staticmethod(parse_config)
