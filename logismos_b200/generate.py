"""Generation from a model folder through the continuous-batching scheduler:

    python -m logismos_b200.generate --model DIR --prompt 5,17,3 --prompt 9,2 --max-new 16
    python -m logismos_b200.generate --model DIR --prompt 5,17,3 --temperature 0.8 --top-k 50 --top-p 0.95 --seed 7

Prompts are token ids (tokenisation stays with the caller). One line of ids per prompt."""
from __future__ import annotations

import argparse
import time
from typing import List, Optional, Sequence

import numpy as np

from .cache import blocks_for
from .registry import Limits, Served, load_model
from .serving import Request, Scheduler, serve


def generate(served: Served, prompts: Sequence[Sequence[int]], max_new: int, chain=None, prefill_token_budget: int = 0) -> List[List[int]]:
    """The continuations of all prompts, in order. ``chain``: a ``sampling.DecodeChain`` over the step's device
    logits (executors that expose them); None: greedy."""
    if not 0 < max_new:
        raise ValueError("max_new must be positive")
    n = served.limits.pool_blocks
    lim = served.limits
    sched = Scheduler(n, n, lim.max_seqs, lim.step_tokens, lim.max_seqs, prefill_token_budget=prefill_token_budget, chunked_prefill=True)
    reqs = [Request(i, np.asarray(p, np.uint32), max_new) for i, p in enumerate(prompts)]

    def step(plan):
        tokens = served.step(plan)
        if chain is not None:
            tokens = chain.step(served.model.logits_tensor()).cpu().numpy()
        return tokens

    t0 = time.perf_counter()
    serve(step, sched, reqs, lambda: time.perf_counter() - t0)
    return [r.output for r in reqs]


def sampling_chain(temperature: float, top_k: int, top_p: float, min_p: float, seed: int):
    from .sampling import DecodeChain, MinP, MultinomialSampler, TemperatureScale, TopK, TopP
    chain = DecodeChain(MultinomialSampler(seed)).push(TemperatureScale(temperature))
    if top_k:
        chain.push(TopK(top_k))
    if top_p < 1.0:
        chain.push(TopP(top_p))
    if min_p > 0.0:
        chain.push(MinP(min_p))
    return chain


def main(argv: Optional[Sequence[str]] = None):
    ap = argparse.ArgumentParser(prog="generate", description="generate from a model folder")
    ap.add_argument("--model", required=True)
    ap.add_argument("--prompt", action="append", required=True, help="comma-separated token ids; may be given several times")
    ap.add_argument("--max-new", type=int, default=32)
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--max-seqs", type=int, default=16, help="sequences decoded together")
    ap.add_argument("--prefill-budget", type=int, default=4096, help="prompt tokens fed per step")
    ap.add_argument("--temperature", type=float, default=0.0, help="0: greedy")
    ap.add_argument("--top-k", type=int, default=0)
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--min-p", type=float, default=0.0)
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--device", type=int, default=0)
    a = ap.parse_args(argv)
    prompts = [[int(t) for t in p.split(",")] for p in a.prompt]
    lifetime = sorted((16 * blocks_for(len(p) + a.max_new) for p in prompts), reverse=True)
    seqs = min(a.max_seqs, len(prompts))
    limits = Limits(sum(lifetime[:seqs]), seqs, max_step_tokens=a.prefill_budget + seqs)
    served = load_model(a.model, limits, a.dtype, a.device, compile_missing=True)
    chain = sampling_chain(a.temperature, a.top_k, a.top_p, a.min_p, a.seed) if a.temperature > 0 else None
    for out in generate(served, prompts, a.max_new, chain, a.prefill_budget):
        print(",".join(str(t) for t in out))
    served.close()


if __name__ == "__main__":
    main()
