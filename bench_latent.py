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


# ---- kernels -------------------------------------------------------------------------------------

def _graph_us(calls, reps=6):
    """Device time per call: the calls (different operands) captured once, replayed."""
    import torch
    from ctypes import c_void_p
    s = torch.cuda.Stream()
    torch.cuda.synchronize()  # the operands were made on another stream
    with torch.cuda.stream(s):
        for c in calls:
            assert c(c_void_p(s.cuda_stream)) == 0
        torch.cuda.synchronize()
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g, stream=s):
            for c in calls:
                c(c_void_p(s.cuda_stream))
        for _ in range(3):
            g.replay()
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record(s)
        for _ in range(reps):
            g.replay()
        e1.record(s)
        torch.cuda.synchronize()
    return 1e3 * e0.elapsed_time(e1) / reps / len(calls)


def kernel_table(z, peaks, T=4096, seqs=64, ctx=8192):
    """Every kernel of the latent-attention decoder at one size, and the like kernel of the int4 decoder, each against
    its roofline (the slower of bytes over the measured copy bandwidth and FLOPs over the measured bf16 peak).
    Operands rotate over copies that exceed L2 together."""
    import ctypes as C
    import torch
    from logismos_b200 import ops
    from logismos_b200._lib import lib
    dev = "cuda"
    P = lambda t: C.c_void_p(t.data_ptr() if t is not None else 0)
    st = torch.zeros(1, dtype=torch.int32, device=dev)
    H, heads, D, Q, R, F = z["width"], z["heads"], z["dim"], z["q_rank"], z["kv_rank"], z["ff"]
    HD = heads * D
    rows = []
    bf = lambda *s: (torch.randn(s, device=dev, dtype=torch.bfloat16) * 0.02)
    f32 = lambda *s: torch.randn(s, device=dev)
    i32 = lambda a: torch.as_tensor(np.asarray(a, np.int32)).to(dev)

    def copies(nbytes):
        return max(2, min(12, int(3e8 // max(nbytes, 1)) + 1))

    def add(phase, name, calls, nbytes, flops=0.0, like=None):
        us = _graph_us(calls)
        if int(st.item()):
            raise RuntimeError("%s / %s: device status 0x%x" % (phase, name, int(st.item())))
        roof = max(nbytes / peaks["hbm"] / 1e3, flops / peaks["tf_burst"] / 1e6)
        rows.append({"phase": phase, "kernel": name, "us": us, "roofline_us": roof, "frac": roof / us, "bound": "hbm" if nbytes / peaks["hbm"] / 1e3 >= flops / peaks["tf_burst"] / 1e6 else "tensor",
                     "like": like})
        return us

    def gemm(phase, name, m, n, k, epi, small=False, like=None):
        """bf16 projection through the tcgen05 kernel or the weight-streaming one."""
        w_bytes = 2.0 * n * k
        nw = copies(w_bytes)
        ws, a = [bf(n, k) for _ in range(nw)], bf(m, k)
        glu = epi in (2, 4)
        cols = n // 2 if glu else n
        out = torch.zeros((m, cols), device=dev, dtype=torch.float32 if epi in (1, 3) else torch.bfloat16)
        bias = torch.zeros(n, device=dev)
        p = (1.702, 7.0, 1.0) if epi == 4 else (0.0, 0.0, 0.0)
        if small:
            calls = [lambda s, w=w: lib.logismos_launch_linear_small_bf16(P(a), P(w), P(bias), P(out), m, n, k, k, cols, 1, 0, 0, 0, epi, *p, s) for w in ws]
        else:
            calls = [lambda s, w=w: lib.logismos_launch_linear_t_act_bf16(P(a), P(w), P(bias), P(out), m, n, k, k, cols, epi | 0x100, *p, P(st), s) for w in ws]
        add(phase, name, calls, w_bytes + 2.0 * m * k + m * cols * out.element_size() * (2 if epi == 1 else 1), 2.0 * m * n * k, like)

    def qlin(phase, name, m, n, k):
        w_bytes = 0.5625 * n * k
        nw = copies(w_bytes)
        codes = [torch.randint(0, 256, (n, k // 2), dtype=torch.uint8, device=dev) for _ in range(nw)]
        scales = [(torch.rand((n, k // 32), device=dev) * 0.02).to(torch.float16) for _ in range(nw)]
        a, acc = bf(m, k), torch.zeros((m, n), device=dev)
        add(phase, name, [lambda s, i=i: lib.logismos_launch_qlinear_int4_g32_acc_f32_static(P(a), P(codes[i]), P(scales[i]), P(acc), m, n, k, k, n, P(st), s) for i in range(nw)],
            w_bytes + 2.0 * m * k + 8.0 * m * n, 2.0 * m * n * k)

    gain = torch.ones(H, device=dev)
    # ---- prefill of T tokens in sequences of 1024
    nq = T // 1024
    hist, coef, x, inv = f32(9, T, H), torch.ones(9, device=dev), f32(T, H), torch.ones(T, device=dev)
    add("prefill", "depth_mix (9 snapshots)", [lambda s: lib.logismos_launch_depth_mix_f32(P(hist), T * H, 9, P(coef), P(None), T, P(x), P(inv), P(None), P(None), 0, T, H, H, 1e-6, P(st), s)] * 2,
        10.0 * T * H * 4, like="rms_norm")
    w4, o1, o2 = torch.ones((4, H), device=dev), bf(T, H), bf(T, H)
    state, slots = torch.zeros((64, 2, 3, H), device=dev), i32(range(seqs))
    zero8, seq_ids, cu = torch.zeros(seqs, dtype=torch.uint8, device=dev), i32(np.repeat(np.arange(nq), 1024)), i32(np.arange(nq + 1) * 1024)
    xs = [f32(T, H) for _ in range(copies(T * H * 4))]
    add("prefill", "norm_conv", [lambda s, y=y: lib.logismos_launch_norm_conv(P(y), P(inv), P(gain), P(w4), P(w4), P(o1), P(o2), 0, P(state), P(slots), P(zero8), P(zero8), P(seq_ids), P(cu), T, H, 4, s)
                                     for y in xs], 8.0 * T * H, like="rms_norm")
    gemm("prefill", "latent projections", T, Q + R, H, 3, like="qkv GEMM")
    raws, pool = [f32(T, Q + R) for _ in range(copies(T * (Q + R) * 4))], bf(seqs * (ctx // 16 + 1), 16, R)
    cq, gq, gc, slot64 = bf(T, Q), torch.ones(Q, device=dev), torch.ones(R, device=dev), torch.randperm(T, device=dev)
    add("prefill", "latent_norm_store", [lambda s, y=y: lib.logismos_launch_latent_norm_store(P(y), Q + R, P(gq), P(gc), P(cq), P(pool), P(slot64), T, Q, Q, R, R, 1e-6, pool.shape[0] * 16, 0, 0, P(None), P(st), s)
                                             for y in raws], 6.0 * T * (Q + R), like="rms_norm")
    gemm("prefill", "queries", T, HD, Q, 0, like="qkv GEMM")
    nblk = 1024 // 16
    tabs = i32(np.random.default_rng(0).permutation(nq * nblk).reshape(nq, nblk))
    kv_lens, tp = i32([1024] * nq), int(lib.logismos_latent_gather_rows(T, nq))
    lat, start = bf(tp, R), i32(np.arange(nq) * 1024)
    pools = [bf(nq * nblk, 16, R) for _ in range(copies(2 * T * R * 4))]
    add("prefill", "latent_gather", [lambda s, y=y: lib.logismos_launch_latent_gather_bf16(P(y), P(tabs), nblk, nq * nblk, P(kv_lens), P(lat), P(start), T, nq, 1024, R, P(st), s) for y in pools],
        4.0 * T * R, like="transpose_v")
    gemm("prefill", "keys (values: the transposed product)", tp, HD, R, 0, like="qkv GEMM")
    qs, ks, vts, att = bf(T, HD), bf(tp, HD), bf(HD, tp), bf(T, HD)
    add("prefill", "attention", [lambda s: lib.logismos_launch_varlen_attention_kv_tc_bf16(P(qs), HD, P(cu), P(kv_lens), P(start), P(ks), P(vts), tp, P(att), HD, T, nq, 1024, heads, heads, D, 0.09, P(None), 0, P(st), s)] * 3,
        2.0 * T * HD * 4, 4.0 * HD * nq * 1024 * 1025 / 2, like="attention")
    gemm("prefill", "gated feed-forward", T, 2 * F, H, 4, like="gate/up GEMM")
    gemm("prefill", "output projection [W_o | W_down]", T, H, HD + F, 1, like="down GEMM")
    # like kernels of the int4 decoder
    KV = HD // 4
    add("prefill", "= rms_norm", [lambda s, y=y: lib.logismos_launch_rms_norm_f32(P(y), P(gain), P(o1), T, H, 1e-6, 0, s) for y in xs], 6.0 * T * H)
    gemm("prefill", "= qkv GEMM", T, HD + 2 * KV, H, 0)
    gemm("prefill", "= gate/up GEMM", T, 2 * F, H, 2)
    gemm("prefill", "= down GEMM", T, H, F, 1)
    qkv = bf(T, HD + 2 * KV)
    scr = torch.empty(lib.logismos_varlen_attention_tc_scratch_bytes(T, nq, heads // 4, D), dtype=torch.uint8, device=dev)
    add("prefill", "= attention (with transpose_v)", [lambda s: lib.logismos_launch_varlen_attention_tc_bf16(P(qkv), P(cu), P(att), P(scr), T, nq, 1024, heads, heads // 4, D, HD + 2 * KV, HD, HD + KV, 1, P(st), s)] * 3,
        2.0 * T * HD * 2 + 4.0 * T * KV, 4.0 * HD * nq * 1024 * 1025 / 2)
    del hist, xs, raws, pools, qs, ks, vts
    # ---- decode of `seqs` sequences with `ctx` tokens each, and of 8 for the projections
    nb = ctx // 16 + 1
    dh = f32(9, seqs, H)
    dx = f32(seqs, H)
    add("decode", "depth_mix_conv_decode (9 snapshots)", [lambda s: lib.logismos_launch_depth_mix_conv_decode(P(dh), seqs * H, 9, P(coef), P(dx), P(gain), P(w4), P(w4), P(o1), P(o2), 0, P(state), P(slots), P(zero8), P(zero8), seqs, H, H, 1e-6, 4, s)] * 4,
        seqs * H * (10 * 4 + 6 * 4 + 4.0), like="rms_norm")
    for m in (8, seqs):
        small = m <= 32
        gemm("decode %d" % m, "latent projections", m, Q + R, H, 3 if small else 1, small, like="int4 linear qkv")
        gemm("decode %d" % m, "queries", m, HD, Q, 0, small, like="int4 linear qkv")
        gemm("decode %d" % m, "gated feed-forward", m, 2 * F, H, 4, m <= 16, like="int4 linear gate/up")
        gemm("decode %d" % m, "output projection [W_o | W_down]", m, H, HD + F, 1, like="int4 linear down")
        gemm("decode %d" % m, "head", m, VOCAB, H, 3, m <= 16, like="int4 linear down")
        wk = [bf(heads, R, D) for _ in range(copies(2 * heads * R * D))]
        aq, oq = bf(m, heads, D), bf(m, heads, R)
        add("decode %d" % m, "latent queries (per head)", [lambda s, w=w: lib.logismos_launch_linear_small_bf16(P(aq), P(w), P(None), P(oq), m, R, D, HD, heads * R, heads, D, R * D, R, 0, 0.0, 0.0, 0.0, s) for w in wk],
            2.0 * heads * (R * D + m * (R + D)), 2.0 * m * heads * R * D, like="int4 linear qkv")
        if m == 8:
            qlin("decode 8", "= int4 linear qkv", m, HD + 2 * KV, H)
            qlin("decode 8", "= int4 linear gate/up", m, 2 * F, H)
            qlin("decode 8", "= int4 linear down", m, H, F)
        else:
            gemm("decode %d" % m, "= qkv GEMM (bf16 copy)", m, HD + 2 * KV, H, 0)
            gemm("decode %d" % m, "= gate/up GEMM (bf16 copy)", m, 2 * F, H, 2)
            gemm("decode %d" % m, "= down GEMM (bf16 copy)", m, H, F, 1)
    cl = torch.full((seqs,), ctx, dtype=torch.int32)
    tab = i32(np.random.default_rng(1).permutation(seqs * nb).reshape(seqs, nb))
    qd, od, cg = bf(seqs, heads, R), bf(seqs, heads, R), cl.to(dev)
    chunk = int(lib.logismos_pick_latent_chunk(C.c_void_p(cl.data_ptr()), seqs, heads))
    off, total = ops.build_decode_chunks(cl, chunk)
    off = off.to(dev)
    scr = torch.empty(lib.logismos_latent_decode_scratch_bytes(total, heads, R), dtype=torch.uint8, device=dev)
    add("decode", "latent_decode + merge (ctx %d)" % ctx, [lambda s: lib.logismos_launch_latent_decode_bf16(P(qd), P(pool), P(tab), P(cg), P(off), P(od), P(scr), seqs, total, chunk, nb, seqs * nb, heads, R, 0.05, P(None), 0, P(None), 0, 0, P(st), s)] * 3,
        seqs * (ctx * R * 2.0 + heads * R * 4.0), 4.0 * seqs * ctx * heads * R, like="paged_decode")
    del pool
    nkv = heads // 4
    kp, vp = bf(seqs * nb, 16, nkv * D), bf(seqs * nb, 16, nkv * D)
    qp, op = bf(seqs, HD), bf(seqs, HD)
    pc = ops.pick_decode_chunk(cl, nkv, D)
    off2, total2 = ops.build_decode_chunks(cl, pc)
    off2 = off2.to(dev)
    scr2 = torch.empty(lib.logismos_paged_decode_scratch_bytes(total2, heads, D), dtype=torch.uint8, device=dev)
    add("decode", "= paged_decode + merge (ctx %d)" % ctx, [lambda s: lib.logismos_launch_paged_attention_decode_bf16(P(qp), P(kp), P(vp), P(None), P(None), P(tab), P(cg), P(off2), P(op), P(scr2), P(st), seqs, total2, pc, nb, seqs * nb, heads, nkv, D, s)] * 3,
        seqs * ctx * nkv * D * 4.0, 4.0 * seqs * ctx * HD)
    dxs = f32(seqs, H)
    add("decode", "= rms_norm", [lambda s: lib.logismos_launch_rms_norm_f32(P(dxs), P(gain), P(o1), seqs, H, 1e-6, 0, s)] * 4, 6.0 * seqs * H)
    return rows
