"""Replays a given batch schedule through a model, step by step, and writes logits: no sampling, no policy,
the engine's own step, cache blocks and state slots (command line: ``bin/trace_run``)."""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, List, Tuple

import numpy as np

from .cache import BlockAllocator, SlotAllocator
from .registry import Limits, Served, UnsupportedDtype, load_model
from .serving import StepPlan

LIVE_REQUESTS = 4


class Replay:
    """Live requests of a schedule: what each holds in the cache, and the packed step of its next tokens."""

    def __init__(self, served: Served):
        self.served = served
        n = served.limits.pool_blocks
        self.blocks, self.slots = BlockAllocator(n, n), SlotAllocator(served.limits.max_seqs)
        self.cached: Dict[str, int] = {}

    def step(self, entries: List[dict]) -> np.ndarray:
        """Runs the tokens of all entries as one batch; the logits at their wanted places, fp32 [wanted, vocab]."""
        ids, cached, new, tables, slots, want = [], [], [], [], [], []
        entries = [e for e in entries if e["tokens"]]
        for e in entries:
            rid, toks = e["id"], e["tokens"]
            done = self.cached.get(rid, 0)
            want.extend(len(ids) + int(p) for p in e["want"])
            ids.extend(int(t) for t in toks)
            cached.append(done)
            new.append(len(toks))
            self.cached[rid] = done + len(toks)
            tables.append(self.blocks.ensure(rid, done + len(toks)))
            slots.append(self.slots.get(rid))
        if ids:
            plan = StepPlan(np.asarray(ids, np.uint32), np.asarray(cached, np.int32), np.asarray(new, np.int32), np.stack(tables),
                            np.asarray(slots, np.int32), [e["id"] for e in entries], sum(n == 1 for n in new), sum(n for n in new if n > 1))
            self.served.step(plan, out_rows=want)
        return self.served.model.last_logits() if want else np.empty((0, self.served.vocab), np.float32)

    def end(self, rid: str):
        self.blocks.release(rid)
        self.slots.release(rid)
        self.cached.pop(rid, None)


def run(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay batch steps from standard input (one JSON object a line) and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold together")
    ap.add_argument("--device", type=int, default=0)
    a = ap.parse_args(argv)
    limits = Limits(a.max_tokens, LIVE_REQUESTS, max_out_rows=a.max_tokens)
    try:
        served = load_model(a.model, limits, a.dtype, a.device, compile_missing=True)
    except UnsupportedDtype as e:
        print(e, file=sys.stderr)
        return 3
    replay = Replay(served)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = replay.step(s["entries"])
        if logits.shape[0]:
            logits.astype("<f4").tofile(os.path.join(a.out, f"{s['step']}.f32"))
        for rid in s["end"]:
            replay.end(rid)
        print(f"done {s['step']}", flush=True)
    served.close()
    return 0
