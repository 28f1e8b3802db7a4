"""What the executors of decoder steps with per-sequence state slots have in common over the C ABI: the packed
step, logits, diagnostics. A subclass names its entry points (``lg_<prefix>_*``) and creates the handle."""
from __future__ import annotations

import ctypes as C
from typing import Sequence

import numpy as np

from ._lib import lib
from .embed import ComputeError, InputTooLong

_vp = C.c_void_p


def bits_pointer(a: np.ndarray) -> int:
    """Address of an array of bfloat16 bit patterns."""
    assert a.dtype == np.uint16 and a.flags["C_CONTIGUOUS"]
    return a.ctypes.data


class SlotExecutor:
    prefix = ""

    def _fn(self, name):
        return getattr(lib, f"lg_{self.prefix}_{name}")

    def _adopt(self, rc: int, handle, cfg: dict, max_blocks: int, max_step_tokens: int, max_step_seqs: int, device: int, dtype: str):
        if rc:
            raise (IOError if rc == 5 else ComputeError)(lib.lg_last_error().decode())
        self._h, self.cfg, self.max_blocks, self.device, self.dtype = handle, cfg, max_blocks, device, dtype
        self.max_step_tokens, self.max_step_seqs, self._n_out = max_step_tokens, max_step_seqs, 0

    def close(self):
        if getattr(self, "_h", None):
            self._fn("destroy")(self._h)
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
        rc = self._fn("step")(self._h, P(ids), P(cached), P(new), n, P(tables), P(slots), None if rows is None else P(rows), n_out, P(out))
        if rc:
            raise (InputTooLong if rc == 1 else ComputeError)(lib.lg_last_error().decode())
        self._n_out, self._n_tokens = n_out, ids.size
        return out[:n_out]

    def replay_device(self, stream_ptr: int):
        if self._fn("replay_device")(self._h, _vp(stream_ptr)):
            raise ComputeError(lib.lg_last_error().decode())

    def last_logits(self) -> np.ndarray:
        """fp32 [rows asked for, vocab]."""
        out = np.empty((self._n_out, self.cfg["vocab"]), np.float32)
        if self._fn("last_logits")(self._h, self._n_out, out.ctypes.data_as(_vp)):
            raise ComputeError(lib.lg_last_error().decode())
        return out

    def logits_tensor(self):
        """The same as a CUDA tensor over the executor's own buffer (overwritten by the next step): the input
        of ``sampling.DecodeChain``."""
        import torch
        shape = (self._n_out, self.cfg["vocab"])
        view = type("_View", (), {"__cuda_array_interface__": {"shape": shape, "typestr": "<f4", "version": 3,
                                                               "data": (int(self._fn("logits_device")(self._h)), False)}})()
        return torch.as_tensor(view, device=f"cuda:{self.device}")

    def snapshot(self, j: int) -> np.ndarray:
        """The residual stream of the last step at stage j (0: the embedding), fp32 [tokens, hidden]."""
        out = np.empty((self._n_tokens, self.cfg["hidden"]), np.float32)
        if self._fn("snapshot")(self._h, j, self._n_tokens, out.ctypes.data_as(_vp)):
            raise ComputeError(lib.lg_last_error().decode())
        return out

    def launches_last_step(self) -> int:
        return int(self._fn("launches_last_step")(self._h))

    def device_status(self) -> int:
        return int(self._fn("device_status")(self._h))
