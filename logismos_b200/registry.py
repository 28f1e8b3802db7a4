"""Decoder models by the architecture their config.json names: what a model folder is loaded with.

A folder holds config.json and model.safetensors. ``load_model`` reads the first, picks the entry and returns
a ``Served`` model: the executor behind one ``step`` signature (state slots are ignored by executors
without per-sequence state), whatever the architecture."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable, Dict, Optional, Tuple

from .cache import blocks_for


class UnsupportedDtype(ValueError):
    """The architecture has no executor for the requested number format."""


@dataclass(frozen=True)
class Limits:
    """What an executor is sized for."""
    max_tokens: int              # tokens that live sequences hold together
    max_seqs: int                # live sequences (state slots, rows of a step)
    max_step_tokens: int = 0     # tokens of one step (0: max_tokens)
    max_out_rows: int = 0        # rows of logits per step (0: max_seqs)

    @property
    def pool_blocks(self) -> int:
        return blocks_for(self.max_tokens)

    @property
    def step_tokens(self) -> int:
        return self.max_step_tokens or self.max_tokens


@dataclass
class Served:
    architecture: str
    model: object
    takes_slots: bool
    limits: Limits

    @property
    def vocab(self) -> int:
        return self.model.cfg["vocab"]

    def step(self, plan, out_rows=None):
        """One step of a ``serving.StepPlan``; ``out_rows`` selects other tokens than the last of every sequence."""
        args = [plan.ids, plan.cached, plan.new, plan.tables]
        if self.takes_slots:
            args.append(plan.slots)
        if out_rows is not None:
            return self.model.step(*args, out_rows=out_rows)
        return self.model.step(*args)

    def close(self):
        self.model.close()


def _vofosun(folder: str, config: dict, limits: Limits, dtype: str, device: int):
    from .latent import LatentModel
    return LatentModel.load(folder, config, limits.pool_blocks, limits.pool_blocks, limits.step_tokens, limits.max_seqs, limits.max_seqs,
                            device=device, dtype=dtype, max_out_rows=limits.max_out_rows)


def _katadra(folder: str, config: dict, limits: Limits, dtype: str, device: int):
    from .mixer import MixerModel
    return MixerModel.load(folder, config, limits.pool_blocks, limits.pool_blocks, limits.step_tokens, limits.max_seqs, limits.max_seqs,
                           device=device, dtype=dtype, max_out_rows=limits.max_out_rows)


def _vugedra(folder: str, config: dict, limits: Limits, dtype: str, device: int):
    from .vugedra import VugedraModel
    return VugedraModel.load(folder, config, limits.pool_blocks, limits.pool_blocks, limits.step_tokens, limits.max_seqs, limits.max_seqs,
                             device=device, dtype=dtype, max_out_rows=limits.max_out_rows)


def _zetalorn(folder: str, config: dict, limits: Limits, dtype: str, device: int):
    from .zetalorn import ZetalornModel
    return ZetalornModel.load(folder, config, limits.pool_blocks, limits.pool_blocks, limits.step_tokens, limits.max_seqs, limits.max_seqs,
                              device=device, dtype=dtype, max_out_rows=limits.max_out_rows)


def _qwen2(folder: str, config: dict, limits: Limits, dtype: str, device: int):
    from .decoder import DecoderModel
    cfg = dict(vocab=config["vocab_size"], hidden=config["hidden_size"], n_layers=config["num_hidden_layers"],
               n_heads=config["num_attention_heads"], n_kv_heads=config["num_key_value_heads"], intermediate=config["intermediate_size"],
               max_pos=config["max_position_embeddings"], rms_eps=config["rms_norm_eps"], rope_theta=config["rope_theta"])
    return DecoderModel.load(os.path.join(folder, "model.safetensors"), cfg, limits.pool_blocks, limits.pool_blocks, limits.step_tokens,
                             limits.max_seqs, device=device)


@dataclass(frozen=True)
class Entry:
    loader: Callable
    dtypes: Tuple[str, ...]
    takes_slots: bool            # the executor keeps per-sequence state in slots
    build_group: Optional[str]   # the part of the library it needs (build.GROUPS; None: all of it)


REGISTRY: Dict[str, Entry] = {
    "Vofosun": Entry(_vofosun, ("bfloat16", "float32"), True, "latent"),
    "Katadra": Entry(_katadra, ("bfloat16", "float32"), True, "mixer"),
    "Vugedra": Entry(_vugedra, ("bfloat16", "float32"), True, "mixer"),
    "Zetalorn": Entry(_zetalorn, ("bfloat16", "float32"), True, "mixer"),
    "Qwen2ForCausalLM": Entry(_qwen2, ("bfloat16",), False, None),   # int4 weights, bf16 activations
}


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def architecture_of(config: dict) -> str:
    name = config.get("architecture") or (config.get("architectures") or [None])[0]
    if name not in REGISTRY:
        raise ValueError(f"no model of architecture {name!r} (known: {', '.join(sorted(REGISTRY))})")
    return name


def load_model(folder: str, limits: Limits, dtype: str = "bfloat16", device: int = 0, compile_missing: bool = False) -> Served:
    """``compile_missing``: build the part of the library the model needs when it is absent or out of date (for
    command-line tools in a fresh checkout)."""
    config = read_config(folder)
    name = architecture_of(config)
    entry = REGISTRY[name]
    if dtype not in entry.dtypes:
        raise UnsupportedDtype(f"{name} runs in {', '.join(entry.dtypes)}, not in {dtype}")
    if compile_missing:
        from . import build
        build.ensure(entry.build_group)
    return Served(name, entry.loader(folder, config, limits, dtype, device), entry.takes_slots, limits)
