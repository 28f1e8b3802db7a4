"""Decoders over a stack of mixers and feed-forwards of several kinds, over the C ABI (``lg_mixer_*``): weights and the
packed continuous-batching step, and the configuration of the post-norm stack of state-space layers and parallel layers,
attention beside time mixing (Katadra; ``vugedra`` and ``zetalorn`` have the other designs'). The contract is that of the other executors:
a packed step equals running every sequence alone."""
from __future__ import annotations

import ctypes as C
import os
from typing import Optional

from ._lib import lib
from .executor import SlotExecutor, bits_pointer

_vp = C.c_void_p
SSD, PARALLEL, ATTENTION, GLA, LATENT, DIFF, PAIR = range(7)
RELU2, GATED, MIXTURE = range(3)            # feed-forwards
POST_LAYER_NORM, TANH_AROUND, RMS_GATED = range(3)     # norms of the stack
SOFTMAX, SIGMOID = range(2)                 # scores of a router
KINDS = {"mamba2": SSD, "parallel": PARALLEL}

_INT_A = ("kind", "weights_of", "ff", "ssd_heads", "ssd_vdim", "ssd_state", "ssd_groups", "ssd_norm_groups", "ssd_taps", "heads", "kv_heads", "dim", "vdim",
          "bias_rows", "bias_max")
_FLOAT_A = ("scale", "softcap", "temp_coef", "temp_every")
_INT_B = ("tm_heads", "tm_dim", "tm_rank")
_FLOAT_B = ("left_scale", "right_scale")
_INT_C = ("ff_kind", "experts", "identity", "top", "shared_ff", "window", "keep_first", "q_rank", "kv_rank", "rot_dims")
_DOUBLE_C = ("rot_base", "rot_factor", "rot_original", "rot_fast", "rot_slow")
_INT_D = ("rot_halves", "chunked", "pool")
_INT_E = ("lin_heads", "lin_dim", "lin_vdim")
_FLOAT_E = ("glu_alpha", "glu_limit", "glu_shift")
_INT_F = ("scoring", "route_groups", "keep_groups", "no_correction", "file_layer", "pass")


class _LayerCfg(C.Structure):
    _fields_ = [(n, C.c_int32) for n in _INT_A] + [(n, C.c_float) for n in _FLOAT_A] + [(n, C.c_int32) for n in _INT_B] + [(n, C.c_float) for n in _FLOAT_B] + [
        (n, C.c_int32) for n in _INT_C] + [("tau", C.c_float)] + [(n, C.c_double) for n in _DOUBLE_C] + [(n, C.c_int32) for n in _INT_D] + [
        ("diff", C.c_float)] + [(n, C.c_int32) for n in _INT_E] + [("decay", C.POINTER(C.c_double))] + [(n, C.c_float) for n in _FLOAT_E] + [
        (n, C.c_int32) for n in _INT_F]


class _Cfg(C.Structure):
    _fields_ = [(n, C.c_int32) for n in ("vocab", "width", "n_layers")] + [("norm_eps", C.c_float)] + [
        (n, C.c_int32) for n in ("is_f32", "n_pool_blocks", "max_blocks_per_seq", "max_step_tokens", "max_step_seqs", "n_state_slots", "max_out_rows",
                                 "keep_layers")] + [("layers", C.POINTER(_LayerCfg)), ("norm", C.c_int32), ("passes", C.c_int32),
                                                                                  ("logit_scale", C.c_float)]


MIXES = "rkvgw"   # order of the token-shift mixes
_COMMON = ("norm1", "norm1_b", "norm2", "norm2_b", "up", "down")
_SSD = ("in", "conv", "conv_b", "dt_bias", "A_log", "D", "norm", "o")
_LEFT = tuple("left_" + n for n in ("q", "k", "v", "rel", "g", "o"))
_RIGHT = tuple("right_" + n for n in ("r", "k", "v", "g", "w1", "w2", "w0", "u", "norm", "o"))
_TANH = tuple(n + s for n in ("norm1", "norm1b", "norm2", "norm2b") for s in ("", "_b", "_alpha") if n + s not in _COMMON)
_GATED = ("q", "q_b", "q_norm", "k", "k_b", "k_norm", "v", "v_b", "g", "a1", "a2", "a2_b", "dq", "dq_norm", "uq", "dkv", "dkv_norm", "uk", "uv",
          "gate", "router", "correction", "shared_gate", "shared_up", "shared_down")
_PAIRED = ("rg1", "rg1_b", "rg2", "rg2_b", "lq1", "lk1", "lq2", "lk2", "left_q_norm", "left_k_norm", "left_out", "right_q", "right_out")


class _LayerW(C.Structure):
    _fields_ = [(n, _vp) for n in _COMMON + _SSD + _LEFT] + [("mu", _vp * len(MIXES))] + [(n, _vp) for n in _RIGHT + _TANH + _GATED] + [("experts", C.POINTER(_vp))] + [
        (n, _vp) for n in _PAIRED]


class _Weights(C.Structure):
    _fields_ = [(n, _vp) for n in ("embed", "final_norm", "final_norm_b", "head")] + [("layers", C.POINTER(_LayerW)), ("final_norm_alpha", _vp), ("loop_step", _vp)]


def _ssd(m: dict) -> dict:
    return {"ssd_heads": int(m["heads"]), "ssd_vdim": int(m["vdim"]), "ssd_state": int(m["state"]), "ssd_groups": int(m["groups"]),
            "ssd_norm_groups": int(m["norm_groups"]), "ssd_taps": int(m["conv"])}


def _parallel(m: dict) -> dict:
    a, b = m["left"], m["right"]
    temp = a.get("q_temp") or {"coef": 0.0, "every": 1}
    return {"heads": int(a["heads"]), "kv_heads": int(a["kv_heads"]), "dim": int(a["dim"]), "vdim": int(a["vdim"]), "bias_max": int(a["bias_max"]),
            "scale": float(a["scale"]), "softcap": float(a.get("softcap") or 0.0), "temp_coef": float(temp["coef"]), "temp_every": float(temp["every"]),
            "tm_heads": int(b["heads"]), "tm_dim": int(b["dim"]), "left_scale": float(m["left_scale"]), "right_scale": float(m["right_scale"])}


def weights_owner(entries: list, i: int) -> int:
    """The layer whose tensors layer i of a config.json uses, itself or at the end of its weights_of."""
    owner, seen = i, set()
    while entries[owner].get("weights_of") is not None:
        if owner in seen:
            raise ValueError(f"layer {i}: weights_of leads to no layer with tensors of its own")
        seen.add(owner)
        owner = int(entries[owner]["weights_of"])
        if not 0 <= owner < len(entries):
            raise ValueError(f"layer {i}: weights_of names no layer")
    return owner


def check_shared(layers: list):
    for i, y in enumerate(layers):
        if {**layers[y["weights_of"]], "weights_of": 0} != {**y, "weights_of": 0}:
            raise ValueError(f"layer {i}: differs from the layer whose tensors it uses")


def parse_config(config: dict) -> dict:
    """config.json of a Katadra model -> the executor's configuration; the rows of the bias tables (``bias_rows``) and
    the rank of the decays (``tm_rank``) are the tensors' own. Raises ValueError for what the design does not have."""
    layers = []
    for i, lc in enumerate(config["layers"]):
        if lc["type"] not in KINDS:
            raise ValueError(f"layer {i}: no mixer of type {lc['type']!r}")
        mlp = lc.get("mlp")
        if mlp and mlp["kind"] != "dense":
            raise ValueError(f"layer {i}: no feed-forward of kind {mlp['kind']!r}")
        kind = KINDS[lc["type"]]
        layers.append({"kind": kind, "weights_of": weights_owner(config["layers"], i), "ff": int(mlp["ff"]) if mlp else 0,
                       **(_parallel if kind == PARALLEL else _ssd)(lc["mixer"])})
    check_shared(layers)
    return {"vocab": int(config["vocab"]), "hidden": int(config["width"]), "n_layers": len(layers), "norm_eps": float(config["norm"]["eps"]), "layers": layers}


class MixerModel(SlotExecutor):
    """``weights``: dict of bf16 bit patterns (uint16 arrays) embed, final_norm, final_norm_b, head (tanh norms: also
    final_norm_alpha; a gated RMS stack: no final_norm_b, with repeated layers loop_step) and ``layers``: per layer a dict (empty for a layer that uses another's tensors) with the tensors of
    lg_mixer_layer_weights_t that its kind has, by name; ``mu`` is a list of five arrays in the order r, k, v, g, w and
    ``experts`` one of gate, up, down of every expert. ``dtype`` "bfloat16" serves, "float32" computes everything in fp32.
    With ``keep_layers`` ``snapshot(j)`` is the stream before layer j."""

    prefix = "mixer"
    parse = staticmethod(parse_config)

    def __init__(self, cfg: dict, weights: Optional[dict], n_pool_blocks: int, max_blocks_per_seq: int, max_step_tokens: int, max_step_seqs: int,
                 n_state_slots: int, device: int = 0, dtype: str = "bfloat16", max_out_rows: int = 0, keep_layers: bool = False,
                 path: Optional[str] = None):
        if dtype not in ("bfloat16", "float32"):
            raise ValueError(f"dtype {dtype!r}: bfloat16 or float32")
        n = cfg["n_layers"]
        lc = (_LayerCfg * max(1, n))()
        for i, y in enumerate(cfg["layers"]):
            lc[i] = _LayerCfg(**{k: v for k, v in y.items() if k != "decay"})
            if y.get("decay"):
                lc[i].decay = (C.c_double * len(y["decay"]))(*y["decay"])
            if weights is not None and weights["layers"][i]:
                w = weights["layers"][i]
                if y["kind"] == PARALLEL:
                    lc[i].bias_rows, lc[i].tm_rank = w["left_rel"].shape[0], w["right_w1"].shape[0]
                elif y["kind"] == GLA:
                    lc[i].tm_rank = w["a1"].shape[0]
        c = _Cfg(cfg["vocab"], cfg["hidden"], n, cfg["norm_eps"], int(dtype == "float32"), n_pool_blocks, max_blocks_per_seq, max_step_tokens, max_step_seqs,
                 n_state_slots, max(max_out_rows, max_step_seqs), int(keep_layers), lc, cfg.get("norm", POST_LAYER_NORM), cfg.get("passes", 0), cfg.get("logit_scale", 1.0))
        h = _vp()
        if path is not None:
            rc = lib.lg_mixer_load(device, str(path).encode(), C.byref(c), C.byref(h))
        else:
            lw, keep = (_LayerW * max(1, n))(), []
            for i, y in enumerate(weights["layers"]):
                for name, value in y.items():
                    if name == "mu":
                        lw[i].mu = (_vp * len(MIXES))(*[bits_pointer(a) for a in value])
                    elif name == "experts":
                        keep.append((_vp * len(value))(*[bits_pointer(a) for a in value]))
                        lw[i].experts = C.cast(keep[-1], C.POINTER(_vp))
                    else:
                        setattr(lw[i], name, bits_pointer(value))
            w = _Weights(layers=lw)
            for k in ("embed", "final_norm", "final_norm_b", "final_norm_alpha", "head", "loop_step"):
                if k in weights:
                    setattr(w, k, bits_pointer(weights[k]))
            rc = lib.lg_mixer_create(device, C.byref(c), C.byref(w), C.byref(h))
        self._adopt(rc, h, cfg, max_blocks_per_seq, max_step_tokens, max_step_seqs, device, dtype)

    @classmethod
    def load(cls, path: str, config: dict, n_pool_blocks: int, max_blocks_per_seq: int, max_step_tokens: int, max_step_seqs: int, n_state_slots: int,
             device: int = 0, dtype: str = "bfloat16", max_out_rows: int = 0, keep_layers: bool = False) -> "MixerModel":
        """From a model folder (its config.json already read): tensor accounting in the native loader."""
        return cls(cls.parse(config), None, n_pool_blocks, max_blocks_per_seq, max_step_tokens, max_step_seqs, n_state_slots, device, dtype, max_out_rows,
                   keep_layers, path=os.path.join(path, "model.safetensors"))
