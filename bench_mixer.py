"""Prefill and decode throughput of the Katadra decoder (state-space layers, and attention beside time mixing) at
sizes that resemble real layers, beside the hybrid decoder (gated delta rule and gated attention, int4 weights) at
equal width, depth, attention heads and feed-forward (`bench.py --workload mixer`).

Random weights, bf16 (the hybrid's: int4 group-32, with its bf16 copies). Every fourth layer of the Katadra stack is
a parallel layer with a feed-forward, the others are state-space layers without one; the hybrid has a feed-forward in
every layer and full attention in every fourth. Contexts are built by real chunked prefill steps through the same
executor. A step's device work is replayed and timed with CUDA events; the host-buffer entry point is timed around the
same step. Every layer's weights, the states and the cache of all contexts exceed L2 together."""
from __future__ import annotations

import ctypes as C
import time

import numpy as np

from bench_latent import VOCAB, _graph_us

# width, layers; state-space heads x vdim, state, groups; attention heads, key heads, dim; time-mixing heads x dim, rank; feed-forward
SIZES = {
    "1024x16": dict(width=1024, layers=16, sh=32, sv=64, state=128, groups=1, heads=8, kv=2, dim=128, th=16, td=64, rank=64, ff=4096),
    "2048x16": dict(width=2048, layers=16, sh=64, sv=64, state=128, groups=8, heads=16, kv=4, dim=128, th=32, td=64, rank=64, ff=8192),
    "4096x8": dict(width=4096, layers=8, sh=128, sv=64, state=128, groups=8, heads=32, kv=8, dim=128, th=64, td=64, rank=128, ff=14336),
}
FAR, BIAS_ROWS = 1024, 32


def mixer_config(z, vocab=VOCAB):
    ssd = {"kind": 0, "ff": 0, "ssd_heads": z["sh"], "ssd_vdim": z["sv"], "ssd_state": z["state"], "ssd_groups": z["groups"], "ssd_norm_groups": z["groups"], "ssd_taps": 4}
    par = {"kind": 1, "ff": z["ff"], "heads": z["heads"], "kv_heads": z["kv"], "dim": z["dim"], "vdim": z["dim"], "bias_max": FAR, "scale": z["dim"] ** -0.5,
           "softcap": 30.0, "temp_coef": 0.1, "temp_every": 1024.0, "tm_heads": z["th"], "tm_dim": z["td"], "left_scale": 1.0, "right_scale": 1.0}
    return {"vocab": vocab, "hidden": z["width"], "n_layers": z["layers"], "norm_eps": 1e-6,
            "layers": [dict(par if i % 4 == 1 else ssd, weights_of=i) for i in range(z["layers"])]}


def mixer_weights(cfg, z, seed):
    """Layers of one kind share their host arrays (every layer still has its own copy on the device)."""
    rng = np.random.Generator(np.random.PCG64(seed))

    def bits(a):
        return (np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype(np.uint16)

    def mat(n, k, gain=1.0):
        return bits(rng.standard_normal((n, k), dtype=np.float32) * np.float32(gain / np.sqrt(k)))

    H, F, inner, gn = cfg["hidden"], z["ff"], z["sh"] * z["sv"], z["groups"] * z["state"]
    ones, zeros = lambda n: bits(np.ones(n)), lambda n: bits(np.zeros(n))
    norm = {"norm1": ones(H), "norm1_b": zeros(H)}
    ssd = dict(norm, **{"in": mat(2 * inner + 2 * gn + z["sh"], H), "conv": mat(inner + 2 * gn, 4), "conv_b": zeros(inner + 2 * gn),
                        "dt_bias": bits(rng.uniform(-4, 0, z["sh"])), "A_log": bits(rng.uniform(-1, 1, z["sh"])), "D": ones(z["sh"]), "norm": ones(inner), "o": mat(H, inner)})
    HD, TD = z["heads"] * z["dim"], z["th"] * z["td"]
    par = dict(norm, norm2=ones(H), norm2_b=zeros(H), up=mat(F, H), down=mat(H, F), left_q=mat(HD, H), left_k=mat(z["kv"] * z["dim"], H), left_v=mat(z["kv"] * z["dim"], H),
               left_rel=bits(rng.standard_normal((BIAS_ROWS, z["heads"]))), left_g=mat(HD, H), left_o=mat(H, HD), mu=[bits(np.full(H, 0.5))] * 5,
               right_r=mat(TD, H), right_k=mat(TD, H), right_v=mat(TD, H), right_g=mat(TD, H), right_w1=mat(z["rank"], H), right_w2=mat(TD, z["rank"]),
               right_w0=bits(rng.uniform(-6, -0.5, TD)), right_u=bits(0.3 * rng.standard_normal((z["th"], z["td"]))), right_norm=ones(TD), right_o=mat(H, TD))
    return {"embed": mat(cfg["vocab"], H, np.sqrt(H)), "final_norm": ones(H), "final_norm_b": zeros(H), "head": mat(cfg["vocab"], H),
            "layers": [par if y["kind"] else ssd for y in cfg["layers"]]}


def hybrid_config(z, vocab=VOCAB):
    n = z["width"] // 128
    return dict(vocab=vocab, hidden=z["width"], n_layers=z["layers"], n_heads=z["heads"], n_kv_heads=z["kv"], attn_head_dim=z["dim"], gdn_heads=n, intermediate=z["ff"],
                max_pos=65536, full_attn_interval=4, rms_eps=1e-6, rope_theta=1e7)


class Engine:
    """One executor with contexts of ``seqs`` sequences; `which` is "mixer" or "hybrid"."""

    def __init__(self, which, z, seqs, ctx, step_tokens, device=0, seed=5):
        from logismos_b200.cache import BlockAllocator
        self.seqs, self.ctx = seqs, ctx
        mb = (ctx + 64) // 16 + 1
        pool = seqs * mb + 4
        cfg, self.model = self.make(which, z, pool, mb, step_tokens, seqs, device, seed)
        alloc = BlockAllocator(pool, mb, seed=1)
        self.tables = np.stack([alloc.ensure(i, ctx + 1) for i in range(seqs)])
        self.rng = np.random.Generator(np.random.PCG64(9))
        self.vocab, self.step_tokens = cfg["vocab"], step_tokens

    def make(self, which, z, pool, mb, step_tokens, seqs, device, seed):
        """The configuration and the executor."""
        if which == "mixer":
            from logismos_b200.mixer import MixerModel
            cfg = mixer_config(z)
            return cfg, MixerModel(cfg, mixer_weights(cfg, z, seed), pool, mb, step_tokens, seqs, seqs, device=device)
        from logismos_b200.hybrid import HybridModel, random_int4_weights
        cfg = hybrid_config(z)
        return cfg, HybridModel(cfg, random_int4_weights(cfg, seed), pool, mb, step_tokens, seqs, seqs, device=device)

    def step(self, idx, cached, new):
        ids = self.rng.integers(0, self.vocab, int(sum(new)), dtype=np.uint32)
        self.args = [ids, np.asarray(cached, np.int32), np.asarray(new, np.int32), self.tables[idx], np.asarray(idx, np.int32)]
        return self.model.step(*self.args)

    def fill(self, ctx):
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
        for _ in range(iters):
            self.model.step(*self.args)
        return ms, 1e3 * (time.perf_counter() - t0) / iters


def stack_params(which, z):
    """Weights of all layers' matrices."""
    H, F = z["width"], z["ff"]
    n_par = sum(i % 4 == 1 for i in range(z["layers"]))
    if which == "mixer":
        inner, HD, TD = z["sh"] * z["sv"], z["heads"] * z["dim"], z["th"] * z["td"]
        ssd = H * (2 * inner + 2 * z["groups"] * z["state"] + z["sh"]) + H * inner
        par = H * (3 * HD + 2 * z["kv"] * z["dim"]) + 5 * H * TD + z["rank"] * (H + TD) + 2 * H * F
        return n_par * par + (z["layers"] - n_par) * ssd
    QW, KW, GW = z["heads"] * z["dim"], z["kv"] * z["dim"], H
    n_full = z["layers"] // 4
    return z["layers"] * 3 * H * F + n_full * (H * (3 * QW + 2 * KW)) + (z["layers"] - n_full) * (5 * H * GW + 2 * H * (GW // 128))


def decode_bytes(which, z, seqs, ctx, vocab=VOCAB):
    """Algorithmic HBM bytes of one decode step: weights once, cached keys and values, states read and written."""
    wb = 2.0 if which == "mixer" else 0.5625
    n_par = z["layers"] // 4
    kv = n_par * seqs * ctx * 4.0 * z["kv"] * z["dim"]
    if which == "mixer":
        st = 8.0 * seqs * ((z["layers"] - n_par) * z["sh"] * z["sv"] * z["state"] + n_par * z["th"] * z["td"] ** 2)
    else:
        st = 8.0 * seqs * (z["layers"] - n_par) * (z["width"] // 128) * 128 * 128
    return (stack_params(which, z) + vocab * z["width"]) * wb + kv + st


def prefill_flops(which, z, seqs, n):
    """Products of the matrices and of the attention (the recurrences' own products are left out)."""
    return 2.0 * seqs * n * stack_params(which, z) + (z["layers"] // 4) * 4.0 * z["heads"] * z["dim"] * seqs * n * (n + 1) / 2


def measure(sizes, iters, peaks, seqs=(8, 64), ctx=2048, prefill=(4, 1024)):
    import torch
    out = []
    for name in sizes:
        z = SIZES[name]
        row = {"size": name, **z}
        for which in ("mixer", "hybrid"):
            r = {"params": stack_params(which, z)}
            e = Engine(which, z, prefill[0], prefill[1], prefill[0] * prefill[1])
            e.step(list(range(prefill[0])), [0] * prefill[0], [prefill[1]] * prefill[0])
            ms, host = e.time(iters)
            T, fl = prefill[0] * prefill[1], prefill_flops(which, z, *prefill)
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


def kernel_table(z, peaks, T=4096, ctx=8192, batches=(8, 64)):
    """Every kernel of the Katadra decoder at one size, and the like kernel of the hybrid decoder, each against its
    roofline (the slower of bytes over the measured copy bandwidth and FLOPs over the measured bf16 peak). Operands
    rotate over copies that exceed L2 together."""
    import torch
    from logismos_b200 import ops
    from logismos_b200._lib import i32, lib
    from logismos_b200.structs import Groups, ScoreBias, Ssd, TimeMix
    dev = "cuda"
    P = lambda t: C.c_void_p(t.data_ptr() if t is not None else 0)
    A = lambda t: 0 if t is None else t.data_ptr()
    st = torch.zeros(1, dtype=torch.int32, device=dev)
    H, F = z["width"], z["ff"]
    HD, KD, TD, R = z["heads"] * z["dim"], z["kv"] * z["dim"], z["th"] * z["td"], z["rank"]
    inner, gn = z["sh"] * z["sv"], z["groups"] * z["state"]
    ch = inner + 2 * gn
    rows = []
    bf = lambda *s: torch.randn(s, device=dev, dtype=torch.bfloat16) * 0.1
    rf = lambda *s: torch.randn(s, device=dev)
    ints = lambda a: torch.as_tensor(np.asarray(a, np.int32)).to(dev)
    u8 = lambda n: torch.zeros(n, dtype=torch.uint8, device=dev)
    up = lambda v, m: (v + m - 1) // m * m
    keep = []

    def copies(nbytes):
        return max(2, min(12, int(3e8 // max(nbytes, 1)) + 1))

    def add(phase, name, calls, nbytes, flops=0.0, like=None):
        us = _graph_us(calls)
        if int(st.item()):
            raise RuntimeError("%s / %s: device status 0x%x" % (phase, name, int(st.item())))
        roof = max(nbytes / peaks["hbm"] / 1e3, flops / peaks["tf_burst"] / 1e6)
        rows.append({"phase": phase, "kernel": name, "us": us, "roofline_us": roof, "frac": roof / us,
                     "bound": "hbm" if nbytes / peaks["hbm"] / 1e3 >= flops / peaks["tf_burst"] / 1e6 else "tensor", "like": like})

    def gemm(phase, name, m, n, k, epi, small=False, like=None):
        ws, a = [bf(n, k) for _ in range(copies(2.0 * n * k))], bf(m, k)
        glu = epi == 2
        out = torch.zeros((m, n // 2 if glu else n), device=dev, dtype=torch.float32 if epi in (1, 3) else torch.bfloat16)
        if small:
            calls = [lambda s, w=w: lib.logismos_launch_linear_small_bf16(P(a), P(w), P(None), P(out), m, n, k, k, out.shape[1], 1, 0, 0, 0, epi, 0, 0, 0, s) for w in ws]
        else:
            calls = [lambda s, w=w: lib.logismos_launch_linear_t_act_bf16(P(a), P(w), P(None), P(out), m, n, k, k, out.shape[1], epi | 0x100, 0, 0, 0, P(st), s) for w in ws]
        add(phase, name, calls, 2.0 * n * k + 2.0 * m * k + out.numel() * out.element_size() * (2 if epi == 1 else 1), 2.0 * m * n * k, like)

    def grouped(phase, name, m, ends, n_main, cap, like):
        n = ends[-1]
        ws, a = [bf(n, H) for _ in range(copies(2.0 * n * H))], bf(len(ends), m, H)
        out, tail = torch.zeros((m, n_main), device=dev, dtype=torch.bfloat16), torch.zeros((m, n - n_main), device=dev)
        parts = torch.zeros((m, 2 * (n - n_main)), device=dev, dtype=torch.bfloat16) if cap and phase == "prefill" else None
        g = Groups(len(ends), (i32 * 8)(*ends), n_main, A(tail), n - n_main, cap, A(parts))
        keep.append((g, tail, parts))
        if m <= (16 if n * H >= 1 << 23 else 32):
            calls = [lambda s, w=w: lib.logismos_launch_linear_groups_small_bf16(P(a), P(w), P(out), m, n, H, H, n_main, C.byref(g), s) for w in ws]
        else:
            calls = [lambda s, w=w: lib.logismos_launch_linear_groups_tc_bf16(P(a), P(w), P(out), m, n, H, H, n_main, C.byref(g), P(st), s) for w in ws]
        add(phase, name, calls, 2.0 * n * H + 2.0 * a.numel() + 2.0 * m * n_main + 4.0 * tail.numel(), 2.0 * m * n * H, like)

    def qlin(phase, name, m, n, k):
        nw = copies(0.5625 * n * k)
        codes = [torch.randint(0, 256, (n, k // 2), dtype=torch.uint8, device=dev) for _ in range(nw)]
        scales = [(torch.rand((n, k // 32), device=dev) * 0.02).to(torch.float16) for _ in range(nw)]
        a, acc = bf(m, k), torch.zeros((m, n), device=dev)
        add(phase, name, [lambda s, i=i: lib.logismos_launch_qlinear_int4_g32_acc_f32_static(P(a), P(codes[i]), P(scales[i]), P(acc), m, n, k, k, n, P(st), s) for i in range(nw)],
            0.5625 * n * k + 2.0 * m * k + 8.0 * m * n, 2.0 * m * n * k)

    p_main = up(2 * HD + 2 * KD, 128) + 4 * up(TD, 128)
    p_ends = [up(2 * HD + 2 * KD, 128) + i * up(TD, 128) for i in range(5)] + [p_main + up(R, 32)]
    s_main = up(inner + ch, 128)
    s_ends = [s_main + up(z["sh"], 16)]
    gain, mu, w4 = torch.ones(H, device=dev), torch.full((5, H), 0.5, device=dev), torch.full((4, ch), 0.3, device=dev)
    gain_i, gain_t, bias_c = torch.ones(inner, device=dev), torch.ones(TD, device=dev), torch.zeros(ch, device=dev)
    n = z["width"] // 128   # linear-attention heads of the hybrid

    def ssd_args(m, seqs, xbc, proj, dt, y, state, cstate, slots, cu):
        q = [torch.zeros(z["sh"], device=dev), torch.zeros(z["sh"], device=dev), torch.ones(z["sh"], device=dev), u8(seqs), u8(seqs)]
        keep.append(q)
        return Ssd(A(proj), proj.shape[1], A(dt), z["sh"], A(w4), A(bias_c), A(cstate), 4, A(q[0]), A(q[1]), A(q[2]), A(state), A(slots), A(q[3]), A(q[4]), A(cu), A(y),
                       inner, z["sh"], z["groups"], z["state"], z["sv"], A(xbc), ch)

    def tm_args(proj, zz, low, w2, state, seqs, slots, cu, out):
        q = [torch.full((TD,), -2.0, device=dev), torch.full((TD,), 0.3, device=dev), u8(seqs)]
        keep.append(q)
        return TimeMix(A(proj), proj.shape[1], 0, TD, 2 * TD, 3 * TD, A(zz), TD, A(low), R, A(w2), 2 * R, R, A(q[0]), A(q[1]), A(gain_t), A(state), A(slots), A(q[2]), A(cu),
                           A(out), TD, z["th"], z["td"], z["td"], 1.0, 1e-6)

    # ---- prefill of T tokens in sequences of 1024
    nq = T // 1024
    cu, seq_ids, slots = ints(np.arange(nq + 1) * 1024), ints(np.repeat(np.arange(nq), 1024)), ints(range(nq))
    x, ys, h = rf(T, H), [rf(T, H) for _ in range(copies(4 * T * H))], bf(6, T, H)
    shift = torch.zeros((nq, 2, H), device=dev)
    add("prefill", "post_norm", [lambda s, y=y: lib.logismos_launch_post_norm(P(y), 0, P(None), T, P(x), P(gain), P(gain), P(h), 0, T, H, H, 1e-6, P(None), s) for y in ys], 14.0 * T * H, like="rms_norm")
    z8 = u8(64)
    add("prefill", "token_shift", [lambda s, y=y: lib.logismos_launch_token_shift(P(y), P(h), 0, P(mu), 5, P(shift), P(slots), P(z8), P(z8), P(seq_ids), P(cu), T, H, s) for y in ys],
        16.0 * T * H, like="rms_norm")
    grouped("prefill", "projections (parallel layer)", T, p_ends, p_main, 1.0, "linear-attention projections")
    grouped("prefill", "projections (state-space layer)", T, s_ends, s_main, 0.0, "linear-attention projections")
    nblk = 1024 // 16
    tabs, kv_lens = ints(np.random.default_rng(0).permutation(nq * nblk).reshape(nq, nblk)), ints([1024] * nq)
    qkvg = [bf(T, 2 * HD + 2 * KD) for _ in range(copies(2 * T * (2 * HD + 2 * KD)))]
    kp, vpool = bf(nq * nblk, 16, KD), bf(nq * nblk, 16, KD)
    slot64, pos = torch.randperm(T, device=dev), ints(np.tile(np.arange(1024), nq))
    add("prefill", "unit_qk_store", [lambda s, q=q: lib.logismos_launch_unit_qk_store(P(q), q.shape[1], P(kp), P(vpool), P(slot64), P(pos), T, z["heads"], z["kv"], z["dim"], z["dim"], 1e-6, 0.1, 1024.0,
                                                                                     T, 0, P(st), s) for q in qkvg], T * (4.0 * HD + 8.0 * KD), like="rope / rms_norm")
    table = torch.randn((z["heads"], FAR + 1), device=dev)
    sb = [ScoreBias(z["dim"] ** -0.5, 30.0, A(table), FAR, 5.0, 1.2 * z["dim"], A(q) + (HD + 2 * KD) * 2, q.shape[1], 1.0) for q in qkvg]
    att = bf(T, HD)
    scr = torch.empty(lib.logismos_paged_prefix_attention_scratch_bytes(T, nq, z["kv"], z["dim"]), dtype=torch.uint8, device=dev)
    fl_attn = 4.0 * HD * nq * 1024 * 1025 / 2
    add("prefill", "attention, capped and biased (with gather)", [lambda s, q=q, b=b: lib.logismos_launch_bias_attention_prefix_bf16(P(q), q.shape[1], P(cu), P(kv_lens), P(kp), P(vpool), P(tabs), nblk, nq * nblk, P(att), HD, P(scr), T, T,
                                                                                    nq, 1024, 1024, z["heads"], z["kv"], z["dim"], C.byref(b), P(st), s) for q, b in zip(qkvg, sb)], T * (6.0 * HD + 8.0 * KD), fl_attn,
        like="prefix attention")
    add("prefill", "= prefix attention (with gather)", [lambda s, q=q: lib.logismos_launch_paged_prefix_attention_tc_bf16(P(q), q.shape[1], P(cu), P(kv_lens), P(kp), P(vpool), P(tabs), nblk, nq * nblk, P(att), P(scr), T, T,
                                                                                    nq, 1024, 1024, z["heads"], z["kv"], z["dim"], P(st), s) for q in qkvg], T * (4.0 * HD + 8.0 * KD), fl_attn)
    del qkvg
    zz = torch.rand((T, TD), device=dev) * 5.5 - 6.0
    gemm("prefill", "decay projection", T, TD, 2 * R, 3, like="linear-attention projections")
    rkvg = [bf(T, 4 * TD) for _ in range(copies(8 * T * TD))]
    tst, tout = torch.zeros((nq, z["th"], z["td"], z["td"]), device=dev), bf(T, TD)
    ta = [tm_args(q, zz, None, None, tst, nq, slots, cu, tout) for q in rkvg]
    fl_tm = T * z["th"] * (2.0 * z["td"] * z["td"] * 2 + 2.0 * 16 * z["td"] * 2)
    add("prefill", "time_mix_chunk", [lambda s, a=a: lib.logismos_launch_time_mix_chunked_bf16(C.byref(a), nq, s) for a in ta], T * TD * 14.0, fl_tm, like="gdn_chunked")
    del rkvg
    projs = [bf(T, s_main) for _ in range(copies(2 * T * s_main))]
    xbc, dt, y = bf(T, ch), rf(T, z["sh"]), bf(T, inner)
    sst, cst = torch.zeros((nq, z["sh"], z["state"], z["sv"]), device=dev), torch.zeros((nq, 2, 3, ch), device=dev)
    sa = [ssd_args(T, nq, xbc, q, dt, y, sst, cst, slots, cu) for q in projs]
    add("prefill", "ssd_conv", [lambda s, a=a: lib.logismos_launch_ssd_conv(C.byref(a), P(seq_ids), 0, T, 0, 0, s) for a in sa], 4.0 * T * ch, like="rms_norm")
    xbcs = [bf(T, ch) for _ in range(copies(2 * T * ch))]
    sa2 = [ssd_args(T, nq, q, projs[0], dt, y, sst, cst, slots, cu) for q in xbcs]
    fl_ssd = T * z["sh"] * (2.0 * z["state"] * z["sv"] * 2 + 64.0 * (z["state"] + z["sv"]))
    add("prefill", "ssd_chunk", [lambda s, a=a: lib.logismos_launch_ssd_chunked_bf16(C.byref(a), nq, s) for a in sa2], 2.0 * T * (ch + inner), fl_ssd, like="gdn_chunked")
    yi = bf(T, inner)
    add("prefill", "gated_group_norm", [lambda s, q=q: lib.logismos_launch_gated_group_norm(P(yi), inner, P(q), s_main, P(gain_i), P(y), inner, 0, T, z["sh"], z["sv"], z["sv"], z["groups"], 1e-6, s) for q in projs],
        6.0 * T * inner, like="rms_norm")
    del projs, xbcs
    gemm("prefill", "output projection (parallel)", T, H, HD + TD, 3, like="output projection")
    gemm("prefill", "output projection (state-space)", T, H, inner, 3, like="output projection")
    gemm("prefill", "feed-forward up", T, F, H, 5, like="gate/up GEMM")
    gemm("prefill", "feed-forward down", T, H, F, 3, like="down GEMM")
    add("prefill", "= rms_norm", [lambda s, q=q: lib.logismos_launch_rms_norm_f32(P(q), P(gain), P(h), T, H, 1e-6, 0, s) for q in ys], 6.0 * T * H)
    gemm("prefill", "= linear-attention projections", T, 4 * H, H, 0)
    gemm("prefill", "= output projection", T, H, H, 1)
    gemm("prefill", "= gate/up GEMM", T, 2 * F, H, 2)
    gemm("prefill", "= down GEMM", T, H, F, 1)
    gq = [bf(T, 4 * H) for _ in range(copies(8 * T * H))]
    gst, gg, gb, go = torch.zeros((nq, n, 128, 128), device=dev), -torch.rand((T, n), device=dev) * 0.1, torch.rand((T, n), device=dev), bf(T, H)
    gscr = torch.empty(int(lib.logismos_gdn_chunked_scratch_bytes(T, nq, n)), dtype=torch.uint8, device=dev)
    off = lambda t, k: C.c_void_p(t.data_ptr() + 2 * k)
    add("prefill", "= gdn_chunked", [lambda s, q=q: lib.logismos_launch_gdn_chunked(P(gst), off(q, 0), off(q, H), off(q, 2 * H), P(gg), P(gb), P(go), off(q, 3 * H), P(cu), P(slots), P(z8), nq, n, 4 * H, 0.088, P(gscr), T, s)
                                    for q in gq], 10.0 * T * H, T * n * (2.0 * 128 * 128 * 3 + 64.0 * 128 * 5))
    del gq, ys, h
    # ---- decode
    for m in batches:
        ph = "decode %d" % m
        small = lambda nn, kk: m <= (16 if nn * kk >= 1 << 23 else 32)
        grouped(ph, "projections (parallel layer)", m, p_ends, p_main, 1.0, "linear-attention projections")
        grouped(ph, "projections (state-space layer)", m, s_ends, s_main, 0.0, "linear-attention projections")
        gemm(ph, "output projection (parallel)", m, H, HD + TD, 1, like="output projection")
        gemm(ph, "output projection (state-space)", m, H, inner, 1, like="output projection")
        gemm(ph, "feed-forward up", m, F, H, 5, small(F, H), like="gate/up")
        gemm(ph, "feed-forward down", m, H, F, 1, like="down")
        gemm(ph, "head", m, VOCAB, H, 3, small(VOCAB, H), like="gate/up")
        cu1, sl = ints(np.arange(m + 1)), ints(range(m))
        dx, dy, dh, dsh = rf(m, H), rf(m, H), bf(6, m, H), torch.zeros((m, 2, H), device=dev)
        add(ph, "post_norm + shift", [lambda s: lib.logismos_launch_post_norm_shift_decode(P(dy), 0, P(dx), P(gain), P(gain), P(dh), 0, P(mu), 5, P(dsh), P(sl), P(z8), P(z8), m, H, H, 1e-6, s)] * 4,
            m * H * (12.0 + 12.0 + 8.0), like="rms_norm")
        add(ph, "post_norm", [lambda s: lib.logismos_launch_post_norm(P(dy), 0, P(None), m, P(dx), P(gain), P(gain), P(dh), 0, m, H, H, 1e-6, P(None), s)] * 4, m * H * 14.0, like="rms_norm")
        sz = 4.0 * m * z["sh"] * z["state"] * z["sv"]
        ss = [torch.zeros((m, z["sh"], z["state"], z["sv"]), device=dev) for _ in range(copies(sz))]
        dpj, ddt, dyy, dcs = bf(m, s_main), rf(m, z["sh"]), bf(m, inner), torch.zeros((m, 2, 3, ch), device=dev)
        dxb, sid1 = bf(m, ch), ints(range(m))
        da = [ssd_args(m, m, dxb, dpj, ddt, dyy, q, dcs, sl, cu1) for q in ss]
        add(ph, "ssd_conv", [lambda s: lib.logismos_launch_ssd_conv(C.byref(da[0]), P(sid1), 0, m, 1, 0, s)] * 4, m * ch * (4.0 + 24.0), like="rms_norm")
        add(ph, "ssd_step", [lambda s, a=a: lib.logismos_launch_ssd_step(C.byref(a), m, 0, s) for a in da], 2 * sz + 2.0 * m * (ch + inner), like="gdn decode")
        add(ph, "gated_group_norm", [lambda s: lib.logismos_launch_gated_group_norm(P(dyy), inner, P(dpj), s_main, P(gain_i), P(dyy), inner, 0, m, z["sh"], z["sv"], z["sv"], z["groups"], 1e-6, s)] * 4, 6.0 * m * inner, like="rms_norm")
        tz = 4.0 * m * z["th"] * z["td"] ** 2
        tss = [torch.zeros((m, z["th"], z["td"], z["td"]), device=dev) for _ in range(copies(tz))]
        dr, dlow, dw2, dto = bf(m, 4 * TD), rf(m, R), bf(TD, 2 * R), bf(m, TD)
        dta = [tm_args(dr, None, dlow, dw2, q, m, sl, cu1, dto) for q in tss]
        add(ph, "time_mix_step (with decay projection)", [lambda s, a=a: lib.logismos_launch_time_mix_step(C.byref(a), m, 0, s) for a in dta], 2 * tz + m * TD * 10.0 + 2.0 * TD * R, like="gdn decode")
        gz = 4.0 * m * n * 128 * 128
        gss = [torch.zeros((m, n, 128, 128), device=dev) for _ in range(copies(gz))]
        gd, dg, db, dgo = bf(m, 4 * H), -torch.rand((m, n), device=dev), torch.rand((m, n), device=dev), bf(m, H)
        add(ph, "= gdn decode", [lambda s, q=q: lib.logismos_launch_gdn_prefill(P(q), off(gd, 0), off(gd, H), off(gd, 2 * H), P(dg), P(db), P(dgo), off(gd, 3 * H), P(cu1), P(sl), P(z8), m, n, 4 * H, 0.088, 1 | 0x100, s) for q in gss],
            2 * gz + m * H * 10.0)
        acc, pairs = torch.zeros((m, 4 * H + 2 * n), device=dev), torch.zeros(m * n, dtype=torch.int32, device=dev)
        la = torch.zeros(n, device=dev)
        add(ph, "= gdn decode from the accumulator", [lambda s, q=q: lib.logismos_launch_gdn_decode_from_acc(P(q), P(acc), 4 * H + 2 * n, P(la), P(la), P(dgo), P(sl), P(z8), P(pairs), m, n, 0.088, s) for q in gss],
            2 * gz + m * (32.0 * H + 2.0 * H))
        del ss, tss, gss
        if m <= 32:
            qlin(ph, "= linear-attention projections (int4)", m, 4 * H, H)
            qlin(ph, "= output projection (int4)", m, H, H)
            qlin(ph, "= gate/up (int4)", m, 2 * F, H)
            qlin(ph, "= down (int4)", m, H, F)
        else:
            gemm(ph, "= linear-attention projections (bf16 copy)", m, 4 * H, H, 0)
            gemm(ph, "= output projection (bf16 copy)", m, H, H, 1)
            gemm(ph, "= gate/up (bf16 copy)", m, 2 * F, H, 2)
            gemm(ph, "= down (bf16 copy)", m, H, F, 1)
        add(ph, "= rms_norm", [lambda s: lib.logismos_launch_rms_norm_f32(P(dy), P(gain), P(dh), m, H, 1e-6, 0, s)] * 4, 6.0 * m * H)
        nb = ctx // 16 + 1
        kp, vpool = bf(m * nb, 16, KD), bf(m * nb, 16, KD)
        dq, do = bf(m, 2 * HD + 2 * KD), bf(m, HD)
        pos1, slot1 = ints([ctx - 1] * m), torch.randperm(m * nb * 16, device=dev)[:m].contiguous()
        add(ph, "unit_qk_store", [lambda s: lib.logismos_launch_unit_qk_store(P(dq), dq.shape[1], P(kp), P(vpool), P(slot1), P(pos1), m, z["heads"], z["kv"], z["dim"], z["dim"], 1e-6, 0.1, 1024.0, m * nb * 16, 0, P(st), s)] * 4,
            m * (4.0 * HD + 8.0 * KD), like="rms_norm")
        cl = torch.full((m,), ctx, dtype=torch.int32)
        tab, cg = ints(np.random.default_rng(1).permutation(m * nb).reshape(m, nb)), cl.to(dev)
        pc = ops.pick_decode_chunk(cl, z["kv"], z["dim"])
        offs, total = ops.build_decode_chunks(cl, pc)
        offs = offs.to(dev)
        scr2 = torch.empty(lib.logismos_paged_decode_scratch_bytes(total, z["heads"], z["dim"]), dtype=torch.uint8, device=dev)
        b1 = ScoreBias(z["dim"] ** -0.5, 30.0, A(table), FAR, 5.0, 1.2 * z["dim"], A(dq) + (HD + 2 * KD) * 2, dq.shape[1], 1.0)
        add(ph, "decode attention, capped and biased + merge (ctx %d)" % ctx, [lambda s: lib.logismos_launch_bias_attention_decode_bf16(P(dq), dq.shape[1], P(kp), P(vpool), P(tab), P(cg), P(offs), P(do), HD, P(scr2), m, total, pc, nb, m * nb,
                                                                                z["heads"], z["kv"], z["dim"], C.byref(b1), P(st), s)] * 3, m * ctx * KD * 4.0, 4.0 * m * ctx * HD, like="paged_decode")
        add(ph, "= paged_decode + merge (ctx %d)" % ctx, [lambda s: lib.logismos_launch_paged_attention_decode_bf16(P(dq), P(kp), P(vpool), P(None), P(None), P(tab), P(cg), P(offs), P(do), P(scr2), P(st), m, total, pc, nb, m * nb, z["heads"],
                                                                                z["kv"], z["dim"], s)] * 3, m * ctx * KD * 4.0, 4.0 * m * ctx * HD)
        del kp, vpool
    return rows
