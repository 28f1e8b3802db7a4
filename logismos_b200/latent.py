"""Latent-attention decoder (Vofosun: parallel blocks over one norm, input convolutions, depth average,
clamped gated feed-forward, soft-capped head) over the C ABI (``lg_latent_*``): configuration, weights and
the packed continuous-batching step. The contract is that of the other executors: a packed step equals
running every sequence alone."""
from __future__ import annotations

import ctypes as C
import os
from typing import Optional, Sequence

import numpy as np

from ._lib import lib
from .embed import ComputeError, InputTooLong

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


class LatentModel:
    """``weights``: dict of bf16 bit patterns (uint16 arrays) embed, final_norm, head and ``layers``: list of
    dicts norm1, dq, dq_norm, uq, dkv, dkv_norm, uk, uv, o, conv1, dwa and, with a feed-forward, conv2, gate,
    gate_b, up, up_b, down, down_b. ``dtype`` "bfloat16" serves, "float32" computes everything in fp32."""

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
            def ptr(a):
                assert a.dtype == np.uint16 and a.flags["C_CONTIGUOUS"]
                return a.ctypes.data
            lw = (_LayerW * max(1, n))()
            for i, y in enumerate(weights["layers"]):
                for name, _ in _LayerW._fields_:
                    if name in y:
                        setattr(lw[i], name, ptr(y[name]))
            w = _Weights(ptr(weights["embed"]), ptr(weights["final_norm"]), ptr(weights["head"]), lw)
            rc = lib.lg_latent_create(device, C.byref(c), C.byref(w), C.byref(h))
        if rc:
            raise (IOError if rc == 5 else ComputeError)(lib.lg_last_error().decode())
        self._h, self.cfg, self.max_blocks, self.device, self.dtype = h, cfg, max_blocks_per_seq, device, dtype
        self.max_step_tokens, self.max_step_seqs, self._n_out = max_step_tokens, max_step_seqs, 0

    @classmethod
    def load(cls, path: str, config: dict, n_pool_blocks: int, max_blocks_per_seq: int, max_step_tokens: int, max_step_seqs: int,
             n_state_slots: int, device: int = 0, dtype: str = "bfloat16", max_out_rows: int = 0) -> "LatentModel":
        """From a model folder (its config.json already read): tensor accounting in the native loader."""
        return cls(parse_config(config), None, n_pool_blocks, max_blocks_per_seq, max_step_tokens, max_step_seqs, n_state_slots, device,
                   dtype, max_out_rows, os.path.join(path, "model.safetensors"))

    def close(self):
        if getattr(self, "_h", None):
            lib.lg_latent_destroy(self._h)
            self._h = None

    __del__ = close

    def step(self, ids: Sequence[int], cached_lens, new_lens, block_tables, state_slots, out_rows=None) -> np.ndarray:
        """One packed step. Without ``out_rows`` returns the greedy next token of every sequence (uint32
        [n_seqs]); with it (indices into ``ids``, may be empty) the greedy token after each of those."""
        ids = np.ascontiguousarray(ids, dtype=np.uint32)
        cached = np.ascontiguousarray(cached_lens, dtype=np.int32)
        new = np.ascontiguousarray(new_lens, dtype=np.int32)
        tables = np.ascontiguousarray(block_tables, dtype=np.int32)
        slots = np.ascontiguousarray(state_slots, dtype=np.int32)
        n = cached.size
        assert new.size == n and slots.size == n and tables.shape == (n, self.max_blocks) and ids.size == int(new.sum())
        P = lambda a: a.ctypes.data_as(_vp)
        # an empty selection still needs a pointer: NULL selects the last token of every sequence
        rows = None if out_rows is None else np.ascontiguousarray(list(out_rows) + [0], dtype=np.int32)
        n_out = n if rows is None else rows.size - 1
        out = np.empty(max(n_out, 1), np.uint32)
        rc = lib.lg_latent_step(self._h, P(ids), P(cached), P(new), n, P(tables), P(slots), None if rows is None else P(rows), n_out, P(out))
        if rc:
            raise (InputTooLong if rc == 1 else ComputeError)(lib.lg_last_error().decode())
        self._n_out, self._n_tokens = n_out, ids.size
        return out[:n_out]

    def replay_device(self, stream_ptr: int):
        if lib.lg_latent_replay_device(self._h, _vp(stream_ptr)):
            raise ComputeError(lib.lg_last_error().decode())

    def last_logits(self) -> np.ndarray:
        """fp32 [rows asked for, vocab]."""
        out = np.empty((self._n_out, self.cfg["vocab"]), np.float32)
        if lib.lg_latent_last_logits(self._h, self._n_out, out.ctypes.data_as(_vp)):
            raise ComputeError(lib.lg_last_error().decode())
        return out

    def logits_tensor(self):
        """The same as a CUDA tensor over the executor's own buffer (overwritten by the next step): the input
        of ``sampling.DecodeChain``."""
        import torch
        shape = (self._n_out, self.cfg["vocab"])
        view = type("_View", (), {"__cuda_array_interface__": {"shape": shape, "typestr": "<f4", "version": 3,
                                                               "data": (int(lib.lg_latent_logits_device(self._h)), False)}})()
        return torch.as_tensor(view, device=f"cuda:{self.device}")

    def snapshot(self, j: int) -> np.ndarray:
        """X_j of the last step (0 the embedding, i + 1 the result of layer i before averaging), fp32 [tokens, hidden]."""
        out = np.empty((self._n_tokens, self.cfg["hidden"]), np.float32)
        if lib.lg_latent_snapshot(self._h, j, self._n_tokens, out.ctypes.data_as(_vp)):
            raise ComputeError(lib.lg_last_error().decode())
        return out

    def launches_last_step(self) -> int:
        return int(lib.lg_latent_launches_last_step(self._h))

    def device_status(self) -> int:
        return int(lib.lg_latent_device_status(self._h))
