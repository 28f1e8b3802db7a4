"""Latent-attention decoder (Vofosun: parallel blocks over one norm, input convolutions, depth average,
clamped gated feed-forward, soft-capped head) over the C ABI (``lg_latent_*``): configuration, weights and
the packed continuous-batching step. The contract is that of the other executors: a packed step equals
running every sequence alone."""
from __future__ import annotations

import ctypes as C
import os
from typing import Optional

from ._lib import lib
from .executor import SlotExecutor, bits_pointer as ptr

# constants of the design that no configuration carries
NORM_OFFSET, GLU_ALPHA, GLU_SHIFT = 1.0, 1.702, 1.0

_vp = C.c_void_p


class _LayerCfg(C.Structure):
    _fields_ = [(n, C.c_int32) for n in ("heads", "dim", "vdim", "q_rank", "kv_rank", "ff")] + [("scale", C.c_float), ("glu_limit", C.c_float)]


class _Cfg(C.Structure):
    _fields_ = [(n, C.c_int32) for n in ("vocab", "width", "n_layers", "conv_taps")] + [
        (n, C.c_float) for n in ("rms_eps", "norm_offset", "glu_alpha", "glu_shift", "logit_softcap")] + [
        (n, C.c_int32) for n in ("is_f32", "n_pool_blocks", "max_blocks_per_seq", "max_step_tokens", "max_step_seqs", "n_state_slots",
                                 "max_out_rows")] + [("layers", C.POINTER(_LayerCfg))]


_MIX = ("dq", "dq_norm", "uq", "dkv", "dkv_norm", "uk", "uv", "o")
_FF = ("gate", "gate_b", "up", "up_b", "down", "down_b")


class _LayerW(C.Structure):
    _fields_ = [(n, _vp) for n in ("norm1",) + _MIX + _FF + ("conv1", "conv2", "dwa")]


class _Weights(C.Structure):
    _fields_ = [("embed", _vp), ("final_norm", _vp), ("head", _vp), ("layers", C.POINTER(_LayerW))]


def parse_config(config: dict) -> dict:
    """config.json of a Vofosun model -> the executor's configuration. Raises ValueError for what the design
    does not have."""
    layers = []
    for i, lc in enumerate(config["layers"]):
        if lc["type"] != "latent_attention":
            raise ValueError(f"layer {i}: no mixer of type {lc['type']!r}")
        mix, mlp = lc["mixer"], lc.get("mlp")
        if mlp and mlp["kind"] != "dense":
            raise ValueError(f"layer {i}: no feed-forward of kind {mlp['kind']!r}")
        layers.append({"heads": int(mix["heads"]), "dim": int(mix["dim"]), "vdim": int(mix["vdim"]), "q_rank": int(mix["q_rank"]),
                       "kv_rank": int(mix["kv_rank"]), "scale": float(mix["scale"]), "ff": int(mlp["ff"]) if mlp else 0,
                       "glu_limit": float(mlp["limit"]) if mlp else 0.0})
    return {"vocab": int(config["vocab"]), "hidden": int(config["width"]), "n_layers": len(layers), "conv_taps": int(config["canon"]["taps"]),
            "rms_eps": float(config["norm"]["eps"]), "logit_softcap": float(config.get("logit_softcap") or 0.0), "layers": layers}


class LatentModel(SlotExecutor):
    """``weights``: dict of bf16 bit patterns (uint16 arrays) embed, final_norm, head and ``layers``: list of
    dicts norm1, dq, dq_norm, uq, dkv, dkv_norm, uk, uv, o, conv1, dwa and, with a feed-forward, conv2, gate,
    gate_b, up, up_b, down, down_b. ``dtype`` "bfloat16" serves, "float32" computes everything in fp32. ``snapshot(j)`` is X_j (i + 1: the result of
    layer i before averaging)."""

    prefix = "latent"

    def __init__(self, cfg: dict, weights: Optional[dict], n_pool_blocks: int, max_blocks_per_seq: int, max_step_tokens: int,
                 max_step_seqs: int, n_state_slots: int, device: int = 0, dtype: str = "bfloat16", max_out_rows: int = 0,
                 path: Optional[str] = None):
        if dtype not in ("bfloat16", "float32"):
            raise ValueError(f"dtype {dtype!r}: bfloat16 or float32")
        n = cfg["n_layers"]
        lc = (_LayerCfg * max(1, n))()
        for i, y in enumerate(cfg["layers"]):
            lc[i] = _LayerCfg(y["heads"], y["dim"], y["vdim"], y["q_rank"], y["kv_rank"], y["ff"], y["scale"], y["glu_limit"])
        c = _Cfg(cfg["vocab"], cfg["hidden"], n, cfg["conv_taps"], cfg["rms_eps"], NORM_OFFSET, GLU_ALPHA, GLU_SHIFT, cfg["logit_softcap"],
                 int(dtype == "float32"), n_pool_blocks, max_blocks_per_seq, max_step_tokens, max_step_seqs, n_state_slots,
                 max(max_out_rows, max_step_seqs), lc)
        h = _vp()
        if path is not None:
            rc = lib.lg_latent_load(device, str(path).encode(), C.byref(c), C.byref(h))
        else:
            lw = (_LayerW * max(1, n))()
            for i, y in enumerate(weights["layers"]):
                for name, _ in _LayerW._fields_:
                    if name in y:
                        setattr(lw[i], name, ptr(y[name]))
            w = _Weights(ptr(weights["embed"]), ptr(weights["final_norm"]), ptr(weights["head"]), lw)
            rc = lib.lg_latent_create(device, C.byref(c), C.byref(w), C.byref(h))
        self._adopt(rc, h, cfg, max_blocks_per_seq, max_step_tokens, max_step_seqs, device, dtype)

    @classmethod
    def load(cls, path: str, config: dict, n_pool_blocks: int, max_blocks_per_seq: int, max_step_tokens: int, max_step_seqs: int,
             n_state_slots: int, device: int = 0, dtype: str = "bfloat16", max_out_rows: int = 0) -> "LatentModel":
        """From a model folder (its config.json already read): tensor accounting in the native loader."""
        return cls(parse_config(config), None, n_pool_blocks, max_blocks_per_seq, max_step_tokens, max_step_seqs, n_state_slots, device,
                   dtype, max_out_rows, os.path.join(path, "model.safetensors"))
