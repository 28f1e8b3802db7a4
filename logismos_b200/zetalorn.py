"""Configuration of the Zetalorn decoder over the stack-of-mixers executor (``mixer``): RMS norms of one gain ahead of every
sublayer, whose result is gated on its way into the residual; differential attention over chunks, and pooled-window attention
beside linear attention with fixed decays; mixtures of experts with clamped gated units behind a sigmoid router that chooses
among the best groups; a run of layers may be repeated with the same weights."""
from __future__ import annotations

from .mixer import DIFF, MIXTURE, PAIR, RMS_GATED, SIGMOID, MixerModel

KINDS = {"attention": DIFF, "parallel": PAIR}
GLU_ALPHA, GLU_SHIFT = 1.702, 1.0     # a unit is g sigmoid(alpha g) (u + shift)


def _rotation(m: dict, halves: bool) -> dict:
    rot = m.get("rot")
    if not rot:
        return {"rot_dims": 0}
    out = {"rot_dims": int(rot["dims"]), "rot_base": float(rot["base"]), "rot_halves": int(halves)}
    if not 0 <= out["rot_dims"] <= int(m["dim"]):
        raise ValueError(f"{out['rot_dims']} rotated dimensions of {m['dim']}")
    if rot.get("scaling"):
        out["rot_factor"] = float(rot["scaling"]["factor"])
    return out


def _heads(m: dict, halves: bool) -> dict:
    mask = m.get("mask") or {}
    return {"heads": int(m["heads"]), "kv_heads": int(m["kv_heads"]), "dim": int(m["dim"]), "vdim": int(m["vdim"]), "scale": float(m["scale"]),
            "window": int(mask.get("size") or 0), **_rotation(m, halves)}


def _differential(m: dict) -> dict:
    out = _heads(m, halves=False)
    return {**out, "chunked": int(out["window"] > 0), "diff": float(m["diff"])}


def _pair(m: dict) -> dict:
    a, b = m["left"], m["right"]
    decay = [float(d) for d in b["decay"]]
    if len(decay) != int(b["heads"]):
        raise ValueError(f"{len(decay)} decays for {b['heads']} heads")
    return {**_heads(a, halves=True), "pool": int((a.get("mask") or {}).get("pool") or 0), "lin_heads": int(b["heads"]), "lin_dim": int(b["dim"]),
            "lin_vdim": int(b["vdim"]), "decay": decay}


_MIXERS = {DIFF: _differential, PAIR: _pair}


def _feed_forward(mlp) -> dict:
    if not mlp:
        return {"ff": 0}
    if mlp["kind"] != "moe":
        raise ValueError(f"no feed-forward of kind {mlp['kind']!r}")
    r, e = mlp["router"], mlp["expert"]
    groups = r.get("groups") or {"count": 0, "keep": 0}
    if not float(e["limit"]) > 0.0:
        raise ValueError("the limit of the experts' units is positive")
    return {"ff": int(e["ff"]), "ff_kind": MIXTURE, "experts": int(r["experts"]), "top": int(r["top"]), "scoring": SIGMOID, "no_correction": 1,
            "route_groups": int(groups["count"]), "keep_groups": int(groups["keep"]), "glu_alpha": GLU_ALPHA, "glu_limit": float(e["limit"]), "glu_shift": GLU_SHIFT}


def runs(n_layers: int, loop) -> list:
    """(layer, pass that begins with it or None) in the order of execution."""
    if not loop:
        return [(i, None) for i in range(n_layers)]
    a, b, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    if not 0 <= a < b <= n_layers or times < 1:
        raise ValueError(f"no layers {a} .. {b - 1} to run {times} times")
    body = [(i, t if i == a else None) for t in range(times) for i in range(a, b)]
    return [(i, None) for i in range(a)] + body + [(i, None) for i in range(b, n_layers)]


def parse_config(config: dict) -> dict:
    """config.json of a Zetalorn model -> the executor's configuration, a repeated layer listed once per pass. Raises
    ValueError for what the design does not have."""
    parsed = []
    for i, lc in enumerate(config["layers"]):
        if lc["type"] not in KINDS:
            raise ValueError(f"layer {i}: no mixer of type {lc['type']!r}")
        kind = KINDS[lc["type"]]
        try:
            parsed.append({"kind": kind, **_MIXERS[kind](lc["mixer"]), **_feed_forward(lc.get("mlp"))})
        except ValueError as e:
            raise ValueError(f"layer {i}: {e}") from None
    loop, layers, first = config.get("loop"), [], {}
    for at, (i, t) in enumerate(runs(len(parsed), loop)):
        layers.append({**parsed[i], "weights_of": first.setdefault(i, at), "file_layer": i + 1, "pass": 0 if t is None else t + 1})
    return {"vocab": int(config["vocab"]), "hidden": int(config["width"]), "n_layers": len(layers), "norm_eps": float(config["norm"]["eps"]), "norm": RMS_GATED,
            "passes": int(loop["times"]) if loop else 0, "logit_scale": float(config["logit_scale"]), "layers": layers}


class ZetalornModel(MixerModel):
    parse = staticmethod(parse_config)
