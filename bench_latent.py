"""Prefill and decode throughput of the latent-attention decoder (Vofosun) at sizes that resemble real layers,
beside the int4 Qwen2-style decoder at equal width, depth, heads and feed-forward (`bench.py --workload latent`).

Random weights, bf16 (the decoder's: int4 group-32, with its bf16 copies); contexts are built by real chunked
prefill steps through the same executor. A step's device work is replayed and timed with CUDA events; the
host-buffer entry point is timed around the same step. Every layer's weights and the cache of all contexts
exceed L2 together."""
from __future__ import annotations

import time

import numpy as np

# width, layers, heads, head dim, query latent, key/value latent, feed-forward
SIZES = {
    "1024x16": dict(width=1024, layers=16, heads=8, dim=128, q_rank=512, kv_rank=256, ff=4096),
    "2048x16": dict(width=2048, layers=16, heads=16, dim=128, q_rank=1024, kv_rank=512, ff=8192),
    "4096x8": dict(width=4096, layers=8, heads=32, dim=128, q_rank=1536, kv_rank=512, ff=14336),
}
VOCAB = 32768


def latent_config(z, vocab=VOCAB):
    layer = {"heads": z["heads"], "dim": z["dim"], "vdim": z["dim"], "q_rank": z["q_rank"], "kv_rank": z["kv_rank"], "ff": z["ff"],
             "scale": 1.0 / np.sqrt(z["dim"]), "glu_limit": 7.0}
    return {"vocab": vocab, "hidden": z["width"], "n_layers": z["layers"], "conv_taps": 4, "rms_eps": 1e-6, "logit_softcap": 15.0,
            "layers": [layer] * z["layers"]}


def latent_weights(cfg, seed):
    """Layers share their host arrays (every layer still has its own copy on the device); only dwa differs in length."""
    rng = np.random.Generator(np.random.PCG64(seed))

    def bits(a):
        return (np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype(np.uint16)

    def mat(n, k, gain=1.0):
        return bits(rng.standard_normal((n, k), dtype=np.float32) * np.float32(gain / np.sqrt(k)))

    H, y = cfg["hidden"], cfg["layers"][0]
    HD, Q, Rk, F = y["heads"] * y["dim"], y["q_rank"], y["kv_rank"], y["ff"]
    one = dict(norm1=bits(np.zeros(H)), dq=mat(Q, H), dq_norm=bits(np.ones(Q)), uq=mat(HD, Q), dkv=mat(Rk, H), dkv_norm=bits(np.ones(Rk)),
               uk=mat(HD, Rk), uv=mat(HD, Rk), o=mat(H, HD, 0.3), gate=mat(F, H), gate_b=bits(np.zeros(F)), up=mat(F, H), up_b=bits(np.zeros(F)),
               down=mat(H, F, 0.3), down_b=bits(np.zeros(H)), conv1=mat(H, cfg["conv_taps"], 0.3), conv2=mat(H, cfg["conv_taps"], 0.3))
    dwa = lambda i: bits(np.concatenate([np.full(i + 1, 0.02), [1.0]]))
    return {"embed": mat(cfg["vocab"], H, np.sqrt(H)), "final_norm": bits(np.zeros(H)), "head": mat(cfg["vocab"], H),
            "layers": [dict(one, dwa=dwa(i)) for i in range(cfg["n_layers"])]}


def decoder_config(z, vocab=VOCAB):
    return dict(vocab=vocab, hidden=z["width"], n_layers=z["layers"], n_heads=z["heads"], n_kv_heads=z["heads"] // 4, intermediate=z["ff"],
                max_pos=65536, rms_eps=1e-6, rope_theta=1e6)


def decoder_weights(cfg, seed):
    rng = np.random.Generator(np.random.PCG64(seed))
    H, F = cfg["hidden"], cfg["intermediate"]
    KV = cfg["n_kv_heads"] * (H // cfg["n_heads"])

    def q(n, k):
        return (rng.integers(0, 256, (n, k // 2), dtype=np.uint8),
                np.abs(rng.standard_normal((n, k // 32), dtype=np.float32) * np.float32(0.25 / np.sqrt(k))).astype(np.float16))

    one = dict(norm1=np.ones(H, np.float32), norm2=np.ones(H, np.float32), bq=np.zeros(H, np.float32), bk=np.zeros(KV, np.float32),
               bv=np.zeros(KV, np.float32), wq=q(H, H), wk=q(KV, H), wv=q(KV, H), wo=q(H, H), w_gate=q(F, H), w_up=q(F, H), w_down=q(H, F))
    return {"tok_embed": rng.standard_normal((cfg["vocab"], H), dtype=np.float32), "final_norm": np.ones(H, np.float32),
            "lm_head": q(cfg["vocab"], H), "layers": [one] * cfg["n_layers"]}


class Engine:
    """One executor with contexts of ``seqs`` sequences; `which` is "latent" or "decoder"."""

    def __init__(self, which, z, seqs, ctx, step_tokens, device=0, seed=5):
        from logismos_b200.cache import BlockAllocator
        self.which, self.seqs, self.ctx = which, seqs, ctx
        mb = (ctx + 64) // 16 + 1
        pool = seqs * mb + 4
        if which == "latent":
            from logismos_b200.latent import LatentModel
            cfg = latent_config(z)
            self.model = LatentModel(cfg, latent_weights(cfg, seed), pool, mb, step_tokens, seqs, seqs, device=device)
        else:
            from logismos_b200.decoder import DecoderModel
            cfg = decoder_config(z)
            self.model = DecoderModel(cfg, decoder_weights(cfg, seed), pool, mb, step_tokens, seqs, device=device)
        alloc = BlockAllocator(pool, mb, seed=1)
        self.tables = np.stack([alloc.ensure(i, ctx + 1) for i in range(seqs)])
        self.rng = np.random.Generator(np.random.PCG64(9))
        self.vocab, self.step_tokens = cfg["vocab"], step_tokens

    def step(self, idx, cached, new):
        ids = self.rng.integers(0, self.vocab, int(sum(new)), dtype=np.uint32)
        self.args = [ids, np.asarray(cached, np.int32), np.asarray(new, np.int32), self.tables[idx]]
        if self.which == "latent":
            self.args.append(np.asarray(idx, np.int32))
        return self.model.step(*self.args)

    def fill(self, ctx):
        """Prefills every sequence to ctx tokens, whole prompts or chunks of a step."""
        chunk = min(ctx, self.step_tokens)
        per = max(1, self.step_tokens // chunk)
        for s0 in range(0, self.seqs, per):
            idx = list(range(s0, min(self.seqs, s0 + per)))
            for at in range(0, ctx, chunk):
                self.step(idx, [at] * len(idx), [min(chunk, ctx - at)] * len(idx))

    def time(self, iters, warmup=3):
        """(device ms per step, host-entry ms per step) of the last step."""
        import torch
        s = torch.cuda.current_stream()
        for _ in range(warmup):
            self.model.replay_device(s.cuda_stream)
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record(s)
        for _ in range(iters):
            self.model.replay_device(s.cuda_stream)
        e1.record(s)
        torch.cuda.synchronize()
        ms = e0.elapsed_time(e1) / iters
        t0 = time.perf_counter()
        if self.which == "latent":
            idx = self.args[4]
            for _ in range(iters):   # decode positions of the same contexts: the cache row is rewritten each time
                self.model.step(*self.args)
        else:
            for _ in range(iters):
                self.model.step(*self.args)
        return ms, 1e3 * (time.perf_counter() - t0) / iters


def layer_params(which, z):
    H, F, HD = z["width"], z["ff"], z["heads"] * z["dim"]
    if which == "latent":
        return H * (z["q_rank"] + z["kv_rank"]) + HD * z["q_rank"] + 2 * HD * z["kv_rank"] + H * HD + 3 * H * F
    return 2 * H * H + 2 * H * (HD // 4) + 3 * H * F


def prefill_flops(which, z, seqs, n):
    """Products of one step of seqs prompts of n tokens from empty caches (the head runs on one row per prompt)."""
    attn = 4.0 * z["heads"] * z["dim"] * seqs * n * (n + 1) / 2
    return z["layers"] * (2.0 * seqs * n * layer_params(which, z) + attn)


def decode_bytes(which, z, seqs, ctx, vocab=VOCAB):
    """Algorithmic HBM bytes of one decode step: weights once, cache rows of the contexts, residual snapshots."""
    w_bytes = 2.0 if which == "latent" else 0.5625
    row = z["kv_rank"] * 2 if which == "latent" else 2 * (z["heads"] // 4) * z["dim"] * 2
    snaps = sum(2 + i for i in range(z["layers"])) * seqs * z["width"] * 4 if which == "latent" else 0
    head = vocab * z["width"] * w_bytes
    return z["layers"] * (layer_params(which, z) * w_bytes + seqs * ctx * row) + head + snaps


def measure(sizes, iters, peaks, seqs=(8, 64), ctx=2048, prefill=(4, 1024)):
    import torch
    out = []
    for name in sizes:
        z = SIZES[name]
        row = {"size": name, **z}
        for which in ("latent", "decoder"):
            r = {"params_per_layer": layer_params(which, z)}
            e = Engine(which, z, prefill[0], prefill[1], prefill[0] * prefill[1])
            e.step(list(range(prefill[0])), [0] * prefill[0], [prefill[1]] * prefill[0])
            ms, host = e.time(iters)
            T = prefill[0] * prefill[1]
            fl = prefill_flops(which, z, *prefill)
            r["prefill"] = {"tokens": T, "device_ms": ms, "host_ms": host, "tokens_per_s": 1e3 * T / ms, "e2e_tokens_per_s": 1e3 * T / host, "tflops": fl / ms / 1e9,
                            "frac_of_measured_bf16": fl / ms / 1e9 / peaks["tf_sust"], "launches": e.model.launches_last_step()}
            assert e.model.device_status() == 0
            e.model.close()
            r["decode"] = []
            for n in seqs:
                e = Engine(which, z, n, ctx, 4096)
                e.fill(ctx)
                e.step(list(range(n)), [ctx] * n, [1] * n)
                ms, host = e.time(iters)
                by = decode_bytes(which, z, n, ctx)
                r["decode"].append({"seqs": n, "context": ctx, "device_ms": ms, "host_ms": host, "tokens_per_s": 1e3 * n / ms, "e2e_tokens_per_s": 1e3 * n / host,
                                    "gb_per_step": by / 1e9, "gb_per_s": by / ms / 1e6, "frac_of_measured_hbm": by / ms / 1e6 / peaks["hbm"],
                                    "launches": e.model.launches_last_step()})
                assert e.model.device_status() == 0
                e.model.close()
            row[which] = r
            torch.cuda.empty_cache()
        out.append(row)
    return out
