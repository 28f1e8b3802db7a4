"""Prefill and decode throughput of the Vugedra decoder (latent attention, windowed attention and gated linear attention in
turn, each with a mixture of experts) at sizes that resemble real layers, beside the Katadra decoder, whose executor and bf16
weights it shares, at equal width, depth and attention heads (`bench.py --workload vugedra`).

Random weights, bf16. Contexts are built by real chunked prefill steps through the same executor. A step's device work is
replayed and timed with CUDA events; the host-buffer entry point is timed around the same step. Every layer's weights, the
states and the cache of all contexts exceed L2 together."""
from __future__ import annotations

import ctypes as C

import numpy as np

import bench_mixer
from bench_latent import VOCAB, _graph_us

WINDOW, KEEP, EXPERTS, IDENTITY, TOP = 512, 4, 16, 4, 2
# width, layers; heads of both kinds of attention (kv: key heads of the windowed one) of 128; latents; linear-attention heads of gk x gv; expert size
SIZES = {
    "1024x16": dict(width=1024, layers=16, heads=8, kv=2, q_rank=512, kv_rank=256, gh=8, gk=64, gv=128, ff=512),
    "2048x16": dict(width=2048, layers=16, heads=16, kv=4, q_rank=1024, kv_rank=512, gh=16, gk=64, gv=128, ff=1024),
    "4096x8": dict(width=4096, layers=8, heads=32, kv=8, q_rank=1536, kv_rank=512, gh=32, gk=64, gv=128, ff=2048),
}
DIM, NOPE, ROT, RANK = 128, 96, 32, 16   # attention head; unrotated and rotated part of a latent head; rank of the decay
YARN = {"rot_base": 1e4, "rot_factor": 8.0, "rot_original": 4096.0, "rot_fast": 32.0, "rot_slow": 1.0}


def kind_of(i):
    return ("latent", "attention", "gla")[i % 3]


def vugedra_config(z, vocab=VOCAB):
    moe = {"ff": z["ff"], "ff_kind": 2, "experts": EXPERTS, "identity": IDENTITY, "top": TOP, "shared_ff": z["ff"]}
    kinds = {"attention": {"kind": 2, "heads": z["heads"], "kv_heads": z["kv"], "dim": DIM, "vdim": DIM, "scale": DIM ** -0.5, "window": WINDOW, "keep_first": KEEP, "rot_dims": 64, **YARN},
             "gla": {"kind": 3, "heads": z["gh"], "dim": z["gk"], "vdim": z["gv"], "tau": 16.0},
             "latent": {"kind": 4, "heads": z["heads"], "dim": NOPE, "vdim": DIM, "scale": DIM ** -0.5, "q_rank": z["q_rank"], "kv_rank": z["kv_rank"], "rot_dims": ROT, **YARN}}
    return {"vocab": vocab, "hidden": z["width"], "n_layers": z["layers"], "norm_eps": 1e-6, "norm": 1,
            "layers": [dict(kinds[kind_of(i)], **moe, weights_of=i) for i in range(z["layers"])]}


def vugedra_weights(cfg, z, seed):
    """Layers of one kind, and experts, share their host arrays (every one still has its own copy on the device)."""
    rng = np.random.Generator(np.random.PCG64(seed))

    def bits(a):
        return (np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype(np.uint16)

    def mat(n, k, gain=1.0):
        return bits(rng.standard_normal((n, k), dtype=np.float32) * np.float32(gain / np.sqrt(k)))

    H, F, HD, KD = cfg["hidden"], z["ff"], z["heads"] * DIM, z["kv"] * DIM
    ones, zeros = lambda n: bits(np.ones(n)), lambda n: bits(np.zeros(n))
    common = {}
    for n in ("norm1", "norm1b", "norm2", "norm2b"):
        common.update({n: ones(H), n + "_b": zeros(H), n + "_alpha": bits(np.full(1, 0.7))})
    up, down = mat(F, H), mat(H, F)
    common.update(router=mat(EXPERTS + IDENTITY, H), correction=zeros(EXPERTS + IDENTITY), shared_gate=up, shared_up=up, shared_down=down, experts=[up, up, down] * EXPERTS)
    gk, gv, Q, R = z["gh"] * z["gk"], z["gh"] * z["gv"], z["q_rank"], z["kv_rank"]
    kinds = {"attention": dict(common, q=mat(HD, H), q_b=zeros(HD), q_norm=ones(HD), k=mat(KD, H), k_b=zeros(KD), k_norm=ones(KD), v=mat(KD, H), v_b=zeros(KD), g=mat(z["heads"], H),
                               o=mat(H, HD)),
             "gla": dict(common, q=mat(gk, H), k=mat(gk, H), v=mat(gv, H), g=mat(gv, H), a1=mat(RANK, H), a2=mat(gk, RANK), a2_b=bits(np.full(gk, 2.0)), norm=ones(z["gv"]), o=mat(H, gv)),
             "latent": dict(common, dq=mat(Q, H), dq_norm=ones(Q), uq=mat(z["heads"] * (NOPE + ROT), Q), dkv=mat(R + ROT, H), dkv_norm=ones(R), uk=mat(z["heads"] * NOPE, R),
                            uv=mat(HD, R), g=mat(z["heads"], H), o=mat(H, HD))}
    return {"embed": mat(cfg["vocab"], H, np.sqrt(H)), "head": mat(cfg["vocab"], H), "final_norm": ones(H), "final_norm_b": zeros(H), "final_norm_alpha": bits(np.full(1, 0.7)),
            "layers": [kinds[kind_of(i)] for i in range(cfg["n_layers"])]}


class Engine(bench_mixer.Engine):
    def make(self, which, z, pool, mb, step_tokens, seqs, device, seed):
        if which != "vugedra":
            return super().make(which, z, pool, mb, step_tokens, seqs, device, seed)
        from logismos_b200.vugedra import VugedraModel
        cfg = vugedra_config(z)
        return cfg, VugedraModel(cfg, vugedra_weights(cfg, z, seed), pool, mb, step_tokens, seqs, seqs, device=device)


def mixer_params(z, kind):
    """Matrix weights of a mixer."""
    H, HD, KD = z["width"], z["heads"] * DIM, z["kv"] * DIM
    if kind == "attention":
        return H * (2 * HD + 2 * KD + z["heads"])
    if kind == "gla":
        return H * z["gh"] * (2 * z["gk"] + 3 * z["gv"]) + RANK * (H + z["gh"] * z["gk"])
    Q, R = z["q_rank"], z["kv_rank"]
    return H * (Q + R + ROT + z["heads"]) + Q * z["heads"] * (NOPE + ROT) + R * z["heads"] * (NOPE + DIM) + H * HD


def stack_params(z, experts):
    """Matrix weights of all layers with so many routed experts each (the shared one included)."""
    return sum(mixer_params(z, kind_of(i)) + 3 * z["width"] * z["ff"] * (experts + 1) + z["width"] * (EXPERTS + IDENTITY) for i in range(z["layers"]))


def active_experts(tokens=None):
    """Routed experts that a token uses, or that a step of so many tokens touches, by even chances."""
    n = EXPERTS + IDENTITY
    return TOP * EXPERTS / n if tokens is None else EXPERTS * (1.0 - (1.0 - TOP / n) ** tokens)


def decode_bytes(z, seqs, ctx, vocab=VOCAB):
    """Algorithmic HBM bytes of one decode step: weights of what is used once, cached rows that are seen, states."""
    by = 2.0 * (stack_params(z, active_experts(seqs)) + vocab * z["width"])
    for i in range(z["layers"]):
        k = kind_of(i)
        by += seqs * (8.0 * z["gh"] * z["gk"] * z["gv"] if k == "gla" else 2.0 * ctx * (z["kv_rank"] + ROT) if k == "latent" else 4.0 * min(ctx, WINDOW + KEEP) * z["kv"] * DIM)
    return by


def window_pairs(n, size=WINDOW, keep=KEEP):
    """Query-key pairs of a prompt of n tokens."""
    i = np.arange(n)
    return float(np.minimum(i + 1, size + np.minimum(keep, np.maximum(i + 1 - size, 0))).sum())


def prefill_flops(z, seqs, n):
    fl = 2.0 * seqs * n * stack_params(z, active_experts())
    for i in range(z["layers"]):
        k = kind_of(i)
        fl += 4.0 * z["heads"] * DIM * seqs * (window_pairs(n) if k == "attention" else n * (n + 1) / 2 if k == "latent" else 0.0)
    return fl


def katadra_size(z):
    return bench_mixer.SIZES["%dx%d" % (z["width"], z["layers"])]


def measure(sizes, iters, peaks, seqs=(8, 64), ctx=2048, prefill=(4, 1024)):
    import torch
    out = []
    for name in sizes:
        z, kz = SIZES[name], katadra_size(SIZES[name])
        row = {"size": name, **z}
        for which in ("vugedra", "mixer"):
            own = which == "vugedra"
            zz = z if own else kz
            r = {"params": stack_params(z, EXPERTS) if own else bench_mixer.stack_params("mixer", kz), "params_per_token": stack_params(z, active_experts()) if own else bench_mixer.stack_params("mixer", kz)}
            e = Engine(which, zz, prefill[0], prefill[1], prefill[0] * prefill[1])
            e.step(list(range(prefill[0])), [0] * prefill[0], [prefill[1]] * prefill[0])
            ms, host = e.time(iters)
            T, fl = prefill[0] * prefill[1], prefill_flops(z, *prefill) if own else bench_mixer.prefill_flops("mixer", kz, *prefill)
            r["prefill"] = {"tokens": T, "device_ms": ms, "host_ms": host, "tokens_per_s": 1e3 * T / ms, "e2e_tokens_per_s": 1e3 * T / host, "tflops": fl / ms / 1e9,
                            "frac_of_measured_bf16": fl / ms / 1e9 / peaks["tf_sust"], "launches": e.model.launches_last_step()}
            assert e.model.device_status() == 0
            e.model.close()
            r["decode"] = []
            for n in seqs:
                e = Engine(which, zz, n, ctx, 4096)
                e.fill(ctx)
                e.step(list(range(n)), [ctx] * n, [1] * n)
                ms, host = e.time(iters)
                by = decode_bytes(z, n, ctx) if own else bench_mixer.decode_bytes("mixer", kz, n, ctx)
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
    """Every kernel of the Vugedra decoder at one size, and the like kernels ("= ...") of the Katadra decoder, or, for what only
    the latent-attention decoder has, of that one, each against its roofline (the slower of bytes over the measured copy
    bandwidth and FLOPs over the measured bf16 peak). Operands rotate over copies that exceed L2 together."""
    import torch
    from logismos_b200 import ops
    from logismos_b200._lib import check, i32, lib
    from logismos_b200.structs import Groups, LatentRotary, MixtureOut, MoeRoute, ScoreBias, TanhNorm, TimeMix, Window
    dev, rows, keep = "cuda", [], []
    P = lambda t: C.c_void_p(t.data_ptr() if t is not None else 0)
    A = lambda t: 0 if t is None else t.data_ptr()
    st = torch.zeros(1, dtype=torch.int32, device=dev)
    kz = katadra_size(z)
    H, F, heads, kv, HD, KD = z["width"], z["ff"], z["heads"], z["kv"], z["heads"] * DIM, z["kv"] * DIM
    gh, gk, gv, Q, R = z["gh"], z["gk"], z["gv"], z["q_rank"], z["kv_rank"]
    kw, vw = gh * gk, gh * gv
    up = lambda v, m: (v + m - 1) // m * m
    Rp, groups, pairs, hg = up(R + ROT, 64), EXPERTS + 1, TOP + 1, up(heads, 16)
    NL = Q + Rp + hg
    bf = lambda *s: torch.randn(s, device=dev, dtype=torch.bfloat16) * 0.1
    rf = lambda *s: torch.randn(s, device=dev)
    zf = lambda *s: torch.zeros(s, device=dev)
    ints = lambda a: torch.as_tensor(np.asarray(a, np.int32)).to(dev)
    it = lambda *s: torch.zeros(s, dtype=torch.int32, device=dev)
    u8 = lambda n: torch.zeros(n, dtype=torch.uint8, device=dev)

    def copies(nbytes):
        return max(2, min(12, int(3e8 // max(nbytes, 1)) + 1))

    def add(phase, name, calls, nbytes, flops=0.0, like=None):
        us = _graph_us(calls)
        if int(st.item()):
            raise RuntimeError("%s / %s: device status 0x%x" % (phase, name, int(st.item())))
        roof = max(nbytes / peaks["hbm"] / 1e3, flops / peaks["tf_burst"] / 1e6)
        rows.append({"phase": phase, "kernel": name, "us": us, "roofline_us": roof, "frac": roof / us,
                     "bound": "hbm" if nbytes / peaks["hbm"] / 1e3 >= flops / peaks["tf_burst"] / 1e6 else "tensor", "like": like})

    streams = lambda m, n, k: m <= (16 if n * k >= 1 << 23 else 32)

    def gemm(phase, name, m, n, k, epi, like=None):
        """A projection by the route that the executor takes for m rows."""
        ws, a = [bf(n, k) for _ in range(copies(2.0 * n * k))], bf(m, k)
        out = torch.zeros((m, n // 2 if epi == 2 else n), device=dev, dtype=torch.float32 if epi in (1, 3) else torch.bfloat16)
        if epi != 1 and streams(m, n, k):
            calls = [lambda s, w=w: lib.logismos_launch_linear_small_bf16(P(a), P(w), P(None), P(out), m, n, k, k, out.shape[1], 1, 0, 0, 0, epi, 0, 0, 0, s) for w in ws]
        else:
            calls = [lambda s, w=w: lib.logismos_launch_linear_t_act_bf16(P(a), P(w), P(None), P(out), m, n, k, k, out.shape[1], epi | 0x100, 0, 0, 0, P(st), s) for w in ws]
        add(phase, name, calls, 2.0 * n * k + 2.0 * m * k + out.numel() * out.element_size() * (2 if epi == 1 else 1), 2.0 * m * n * k, like)

    def grouped(phase, name, m, n_main, n_tail, parts=False, copies_in=1, like=None):
        n = n_main + n_tail
        if copies_in == 1 and 32 < m <= 512 and up(n, 128) // 128 * (up(m, 128) // 128) <= 74:   # summed over slices of k, then finished
            ws, a, acc = [bf(n, H) for _ in range(copies(2.0 * n * H))], bf(m, H), zf(m, n)
            out, tail = torch.zeros((m, n_main), device=dev, dtype=torch.bfloat16), zf(m, n_tail)
            g = Groups(1, (i32 * 8)(n), n_main, A(tail), n_tail, 0.0, 0, 0)
            keep.append((g, tail))
            both = lambda s, w: lib.logismos_launch_linear_t_act_bf16(P(a), P(w), P(None), P(acc), m, n, H, H, n, 0x101, 0, 0, 0, P(st), s) or lib.logismos_launch_linear_groups_finish(P(acc), P(out), m, n, n, n_main, C.byref(g), s)
            return add(phase, name + " (with finish)", [lambda s, w=w: both(s, w) for w in ws], 2.0 * n * H + 2.0 * m * H + 2.0 * m * n_main + 4.0 * m * n_tail, 2.0 * m * n * H, like)
        ws, a = [bf(n, H) for _ in range(copies(2.0 * n * H))], bf(copies_in, m, H)
        out, tail = torch.zeros((m, n_main), device=dev, dtype=torch.bfloat16), zf(m, n_tail)
        pt = torch.zeros((m, 2 * n_tail), device=dev, dtype=torch.bfloat16) if parts else None
        ends = [n_main // copies_in // 128 * 128 * (i + 1) for i in range(copies_in - 1)] + [n]
        g = Groups(copies_in, (i32 * 8)(*ends), n_main, A(tail), n_tail, 0.0, A(pt), 0)
        keep.append((g, tail, pt))
        if streams(m, n, H):
            calls = [lambda s, w=w: lib.logismos_launch_linear_groups_small_bf16(P(a), P(w), P(out), m, n, H, H, n_main, C.byref(g), s) for w in ws]
        else:
            calls = [lambda s, w=w: lib.logismos_launch_linear_groups_tc_bf16(P(a), P(w), P(out), m, n, H, H, n_main, C.byref(g), P(st), s) for w in ws]
        add(phase, name, calls, 2.0 * n * H + 2.0 * a.numel() + 2.0 * m * n_main + 4.0 * tail.numel(), 2.0 * m * n * H, like)

    ones, table = torch.ones(max(H, HD, Q, Rp), device=dev), rf(ctx + 16, 64)
    norm = TanhNorm(0.7, A(ones), A(ones))
    Y = lambda n: C.byref(n)

    def mixture(ph, m):
        """The router, the experts' products and the sum."""
        few = lib.logismos_moe_streams(m, TOP, EXPERTS, IDENTITY, 1, H, F)
        ld = up(EXPERTS + IDENTITY, 16)
        logits, corr, h = rf(m, ld), zf(ld), bf(m, H)
        wts, prow, ident, off, tok = zf(m, TOP), it(m, pairs), zf(m), it(groups + 1), it(m * pairs)
        counts, pe = it(EXPERTS), it(m, TOP)
        mt = lib.logismos_moe_max_tiles(m, TOP, EXPERTS, 1)
        tiles, nt, gat = it(mt, 4), it(1), bf(m * pairs, H)
        r = MoeRoute(A(logits), ld, 0, A(corr), EXPERTS, IDENTITY, TOP, 1, A(wts), A(prow), A(ident))
        if few:
            r.offsets, r.row_token = A(off), A(tok)
        else:
            r.counts, r.pair_expert, r.tiles, r.n_tiles = A(counts), A(pe), A(tiles), A(nt)
        keep.append((r, logits, corr, wts, prow, ident, off, tok, counts, pe, tiles, nt))
        fused = few and m * (EXPERTS + IDENTITY) * H <= 1 << 22
        if fused:
            wr, arrived = bf(ld, H), it(1)
            r.h, r.w, r.width, r.arrived = A(h), A(wr), H, A(arrived)
            keep.append((wr, arrived))
        else:
            gemm(ph, "router", m, ld, H, 1 if m > 32 else 3, like="latent projections")
        # rows of the experts, and experts that have any
        check(lib.logismos_launch_moe_route(Y(r), m, torch.cuda.current_stream().cuda_stream), "moe_route")
        rows_of = (off[1:] - off[:-1] if few else counts).cpu().numpy()
        n_rows, used = int(rows_of.sum()) + (0 if few else m), int((rows_of > 0).sum()) + (0 if few else 1)
        nw = max(2, min(6, int(3e8 // (6.0 * F * H * groups)) + 1))
        wu, wd = [bf(groups, 2 * F, H) for _ in range(nw)], [bf(groups, H, F) for _ in range(nw)]
        mid, out = bf(m * pairs, F), bf(m * pairs, H)
        ub, ul = 2.0 * used * 2 * F * H + 2.0 * m * H + 2.0 * n_rows * F, 4.0 * n_rows * F * H
        db, dl = 2.0 * used * F * H + 2.0 * n_rows * F + 2.0 * n_rows * H, 2.0 * n_rows * F * H
        if few:
            add(ph, "router and choice of experts" if fused else "choice of experts", [lambda s: lib.logismos_launch_moe_route(Y(r), m, s)] * 4, m * (2.0 * H if fused else ld * 4.0) + 12.0 * m * pairs, like="post_norm")
            ex = 8 if m <= 8 else 16
            add(ph, "experts, gate and up", [lambda s, w=w: lib.logismos_launch_linear_experts_small_bf16(P(h), P(w), P(mid), P(off), P(tok), groups, m, ex, 2 * F, H, H, F, 2, 0, 0, 0, s) for w in wu], ub, ul, "gate/up")
            add(ph, "experts, down", [lambda s, w=w: lib.logismos_launch_linear_experts_small_bf16(P(mid), P(w), P(out), P(off), P(None), groups, m, ex, H, F, F, H, 0, 0, 0, 0, s) for w in wd], db, dl, "down")
        else:
            def choose(s):
                counts.zero_()
                return lib.logismos_launch_moe_route(Y(r), m, s)
            add(ph, "choice of experts (with clearing)", [choose] * 4, m * (ld * 4.0 + 12.0 * pairs), like="post_norm")
            add(ph, "rows by expert", [lambda s: lib.logismos_launch_moe_place(Y(r), P(h), P(gat), H, m, s)] * 4, 2.0 * H * n_rows, like="latent_gather")
            add(ph, "experts, gate and up", [lambda s, w=w: lib.logismos_launch_linear_experts_tc_bf16(P(gat), m * pairs, P(h), m, P(w), P(mid), P(tiles), P(nt), mt, groups, 2 * F, H, H, F, 2, 0, 0, 0, P(st), s) for w in wu], ub, ul, "gate/up")
            add(ph, "experts, down", [lambda s, w=w: lib.logismos_launch_linear_experts_tc_bf16(P(mid), m * pairs, P(None), 0, P(w), P(out), P(tiles), P(nt), mt, groups, H, F, F, H, 0, 0, 0, 0, P(st), s) for w in wd], db, dl, "down")
        del wu, wd
        x, outs = rf(m, H), [bf(m * pairs, H) for _ in range(copies(2.0 * m * pairs * H))]
        mo = [MixtureOut(A(o), A(prow), A(wts), A(ident), pairs, TOP, 0, 0) for o in outs]
        add(ph, "sum of the experts + tanh norms", [lambda s, o=o: lib.logismos_launch_tanh_norm(P(None), 0, Y(o), P(None), m, P(x), Y(norm), P(h), Y(norm), 0, m, H, P(st), s) for o in mo],
            m * H * 12.0 + 2.0 * n_rows * H, like="post_norm")
        gemm(ph, "= gate/up", int(n_rows) // 16 * 16 if m > 512 else m, 2 * F * (1 if m > 512 else 3), H, 2)
        gemm(ph, "= down", int(n_rows) // 16 * 16 if m > 512 else m, H, F * (1 if m > 512 else 3), 3 if m > 512 else 1)

    def gla_args(proj, zz, low, w2, state, seqs, slots, cu, out, mode):
        q = [torch.full((kw,), 2.0, device=dev), torch.ones(max(vw, kw), device=dev), u8(seqs)]
        keep.append(q)
        if mode:
            return TimeMix(A(proj), proj.shape[1], 0, kw, 2 * kw, 2 * kw + vw, A(zz), kw, A(low), 32, A(w2), 64, 32, A(q[0]), 0, A(q[1]), A(state), A(slots), A(q[2]), A(cu), A(out), vw, gh, gv, gk,
                           1.0, 1e-6, 1, gv, 16.0, gk ** -0.5)
        td, th = kz["td"], kz["th"]
        w = td * th
        q += [torch.full((w,), -2.0, device=dev), torch.full((w,), 0.3, device=dev)]
        return TimeMix(A(proj), proj.shape[1], 0, w, 2 * w, 3 * w, A(zz), w, A(low), kz["rank"], A(w2), 2 * kz["rank"], kz["rank"], A(q[3]), A(q[4]), A(q[1]) if w <= q[1].numel() else A(ones), A(state),
                       A(slots), A(q[2]), A(cu), A(out), w, th, td, td, 1.0, 1e-6)

    # ---- prefill of T tokens in sequences of 1024
    ph, nq = "prefill", T // 1024
    cu, slots, pos = ints(np.arange(nq + 1) * 1024), ints(range(nq)), ints(np.tile(np.arange(1024), nq))
    x, ys, h = rf(T, H), [rf(T, H) for _ in range(copies(4 * T * H))], bf(T, H)
    add(ph, "tanh norms + residual", [lambda s, y=y: lib.logismos_launch_tanh_norm(P(y), 0, None, P(None), T, P(x), Y(norm), P(h), Y(norm), 0, T, H, P(st), s) for y in ys], 14.0 * T * H, like="post_norm")
    add(ph, "= post_norm", [lambda s, y=y: lib.logismos_launch_post_norm(P(y), 0, P(None), T, P(x), P(ones), P(ones), P(h), 0, T, H, H, 1e-6, P(None), s) for y in ys], 14.0 * T * H)
    del ys
    a_main, g_main = up(HD + 2 * KD, 128), up(2 * kw + 2 * vw, 128)
    grouped(ph, "projections, attention", T, a_main, hg, like="projections")
    grouped(ph, "projections, linear attention", T, g_main, 32, True, like="projections")
    kmain = up(2 * HD + 2 * KD, 128) + 4 * kz["th"] * kz["td"]
    grouped(ph, "= projections (parallel layer)", T, kmain, up(kz["rank"], 32), True, 6)
    nblk = 1024 // 16
    tabs, kv_lens, slot64 = ints(np.random.default_rng(0).permutation(nq * nblk).reshape(nq, nblk)), ints([1024] * nq), torch.randperm(T, device=dev)
    qkvs = [bf(T, 2 * HD + 2 * KD) for _ in range(copies(2 * T * (2 * HD + 2 * KD)))]
    kp, vpool, att, gate = bf(nq * nblk, 16, KD), bf(nq * nblk, 16, KD), bf(T, HD), rf(T, hg)
    add(ph, "q, k norm + rotation + store", [lambda s, q=q: lib.logismos_launch_qk_norm_rotary_store(P(q), q.shape[1], P(kp), P(vpool), P(slot64), P(pos), T, heads, kv, DIM, DIM, P(ones), P(ones), 1e-6,
                                                                                                    P(table), 64, T, 0, P(st), s) for q in qkvs], T * (4.0 * HD + 8.0 * KD), like="unit_qk_store")
    add(ph, "= unit_qk_store", [lambda s, q=q: lib.logismos_launch_unit_qk_store(P(q), q.shape[1], P(kp), P(vpool), P(slot64), P(pos), T, heads, kv, DIM, DIM, 1e-6, 0.1, 1024.0, T, 0, P(st), s) for q in qkvs],
        T * (4.0 * HD + 8.0 * KD))
    scr = torch.empty(lib.logismos_paged_prefix_attention_scratch_bytes(T, nq, kv, DIM), dtype=torch.uint8, device=dev)
    w = Window(DIM ** -0.5, WINDOW, KEEP, 1, A(gate), hg)
    fl_win, fl_all = 4.0 * HD * nq * window_pairs(1024), 4.0 * HD * nq * 1024 * 1025 / 2
    add(ph, "window attention (with gather)", [lambda s, q=q: lib.logismos_launch_window_attention_prefix_bf16(P(q), q.shape[1], P(cu), P(kv_lens), P(kp), P(vpool), P(tabs), nblk, nq * nblk, P(att), HD, P(scr), T,
                                                                                                            T, nq, 1024, 1024, heads, kv, DIM, Y(w), P(st), s) for q in qkvs], T * (4.0 * HD + 8.0 * KD), fl_win, "attention with gather")
    tb = torch.randn((heads, 1025), device=dev)
    sb = [ScoreBias(DIM ** -0.5, 30.0, A(tb), 1024, 5.0, 1.2 * DIM, A(q) + (HD + 2 * KD) * 2, q.shape[1], 1.0) for q in qkvs]
    add(ph, "= attention, capped and biased (with gather)", [lambda s, q=q, b=b: lib.logismos_launch_bias_attention_prefix_bf16(P(q), q.shape[1], P(cu), P(kv_lens), P(kp), P(vpool), P(tabs), nblk, nq * nblk, P(att), HD,
                                                                                                                             P(scr), T, T, nq, 1024, 1024, heads, kv, DIM, Y(b), P(st), s) for q, b in zip(qkvs, sb)],
        T * (6.0 * HD + 8.0 * KD), fl_all)
    del qkvs
    gemm(ph, "latent projections", T, NL, H, 3, like="latent projections (latent decoder)")
    gemm(ph, "= latent projections (latent decoder)", T, Q + R, H, 3)
    raws, pool, cq = [rf(T, NL) for _ in range(copies(4 * T * NL))], bf(nq * nblk, 16, Rp), bf(T, Q)
    lr = LatentRotary(A(table), A(pos), R, ROT, A(gate), heads, hg)
    add(ph, "latent norms + rotation + store", [lambda s, y=y: lib.logismos_launch_latent_norm_store(P(y), NL, P(ones), P(ones), P(cq), P(pool), P(slot64), T, Q, Q, Rp, R, 1e-6, T, 0, 0, Y(lr), P(st), s) for y in raws],
        T * (6.0 * (Q + R + ROT) + 8.0 * heads), like="latent_norm_store")
    pool2 = bf(nq * nblk, 16, R)
    add(ph, "= latent_norm_store", [lambda s, y=y: lib.logismos_launch_latent_norm_store(P(y), NL, P(ones), P(ones), P(cq), P(pool2), P(slot64), T, Q, Q, R, R, 1e-6, T, 0, 0, None, P(st), s) for y in raws], T * 6.0 * (Q + R))
    del raws
    gemm(ph, "queries", T, HD, Q, 0, like="queries (latent decoder)")
    qs = [bf(T, HD) for _ in range(copies(2 * T * HD))]
    add(ph, "rotation of the queries", [lambda s, q=q: lib.logismos_launch_rotary_heads(P(q), HD, P(pos), T, heads, DIM, NOPE, P(table), ROT, 0, s) for q in qs], 4.0 * T * heads * ROT, like="unit_qk_store")
    tp = lib.logismos_latent_gather_rows(T, nq)
    lat, start, pools = bf(tp, Rp), it(nq), [bf(nq * nblk, 16, Rp) for _ in range(copies(2 * T * Rp))]
    add(ph, "latent gather", [lambda s, y=y: lib.logismos_launch_latent_gather_bf16(P(y), P(tabs), nblk, nq * nblk, P(kv_lens), P(lat), P(start), T, nq, 1024, Rp, P(st), s) for y in pools], 4.0 * T * Rp, like="latent_gather")
    add(ph, "= latent_gather", [lambda s, y=y: lib.logismos_launch_latent_gather_bf16(P(y), P(tabs), nblk, nq * nblk, P(kv_lens), P(lat), P(start), T, nq, 1024, R, P(st), s) for y in pools], 4.0 * T * R)
    del pools
    gemm(ph, "keys; values", tp, HD, Rp, 0, like="keys; values (latent decoder)")
    gemm(ph, "= keys; values (latent decoder)", tp, HD, R, 0)
    kb, vt = bf(tp, HD), bf(HD, tp)
    for name, g, like in (("latent attention", gate, "attention (latent decoder)"), ("= attention (latent decoder)", None, None)):
        add(ph, name, [lambda s, q=q: lib.logismos_launch_varlen_attention_kv_tc_bf16(P(q), HD, P(cu), P(kv_lens), P(start), P(kb), P(vt), tp, P(att), HD, T, nq, 1024, heads, heads, DIM, 0.09, P(g), hg, P(st), s)
                       for q in qs], 8.0 * T * HD, fl_all, like)
    del qs, kb, vt
    gemm(ph, "decay projection", T, up(kw, 128), 64, 3, like="decay projection (parallel layer)")
    gemm(ph, "= decay projection (parallel layer)", T, kz["th"] * kz["td"], 2 * kz["rank"], 3)
    qg, zz, gst, go = [bf(T, g_main) for _ in range(copies(2 * T * g_main))], rf(T, kw) + 2.0, zf(nq, gh, gk, gv), bf(T, vw)
    ga = [gla_args(q, zz, None, None, gst, nq, slots, cu, go, 1) for q in qg]
    add(ph, "gated linear attention", [lambda s, a=a: lib.logismos_launch_time_mix_chunked_bf16(Y(a), nq, s) for a in ga], T * (8.0 * kw + 6.0 * vw), T * gh * (4.0 * gk * gv + 32.0 * (gk + gv)), "time_mix_chunk")
    tdw = kz["th"] * kz["td"]
    rk, z2, tst, to = [bf(T, 4 * tdw) for _ in range(copies(8 * T * tdw))], torch.rand((T, tdw), device=dev) * 5.5 - 6.0, zf(nq, kz["th"], kz["td"], kz["td"]), bf(T, tdw)
    ta = [gla_args(q, z2, None, None, tst, nq, slots, cu, to, 0) for q in rk]
    add(ph, "= time_mix_chunk", [lambda s, a=a: lib.logismos_launch_time_mix_chunked_bf16(Y(a), nq, s) for a in ta], T * tdw * 14.0, T * kz["th"] * (4.0 * kz["td"] ** 2 + 64.0 * kz["td"]))
    del qg, rk
    gemm(ph, "output projection", T, H, HD, 3, like="output projection (parallel layer)")
    gemm(ph, "= output projection (parallel layer)", T, H, HD + tdw, 3)
    mixture(ph, T)
    # ---- decode
    for m in batches:
        ph = "decode %d" % m
        acc = 32 < m
        grouped(ph, "projections, attention", m, a_main, hg, like="projections")
        grouped(ph, "projections, linear attention", m, g_main, 32, like="projections")
        grouped(ph, "= projections (parallel layer)", m, kmain, up(kz["rank"], 32), False, 6)
        gemm(ph, "latent projections", m, NL, H, 1 if acc else 3, like="latent projections (latent decoder)")
        gemm(ph, "= latent projections (latent decoder)", m, Q + R, H, 1 if acc else 3)
        gemm(ph, "queries", m, HD, Q, 0, like="queries (latent decoder)")
        if m <= 16:
            ws, a, xo, ho = [bf(H, HD) for _ in range(copies(2.0 * H * HD))], bf(m, HD), rf(m, H), bf(m, H)
            add(ph, "output projection with tanh norms", [lambda s, w=w: lib.logismos_launch_linear_small_tanh_norm(P(a), P(w), P(xo), Y(norm), P(ho), Y(norm), m, H, HD, HD, H, s) for w in ws],
                2.0 * H * HD + 2.0 * m * HD + 10.0 * m * H, 2.0 * m * H * HD, "output projection (parallel layer)")
            del ws
        gemm(ph, "output projection", m, H, HD, 1, like="output projection (parallel layer)")
        gemm(ph, "= output projection (parallel layer)", m, H, HD + tdw, 1)
        gemm(ph, "head", m, VOCAB, H, 3, like="gate/up")
        mixture(ph, m)
        x, y, h = rf(m, H), rf(m, H), bf(m, H)
        add(ph, "tanh norms + residual", [lambda s: lib.logismos_launch_tanh_norm(P(y), 1, None, P(None), m, P(x), Y(norm), P(h), Y(norm), 0, m, H, P(st), s)] * 4, 18.0 * m * H, like="post_norm")
        add(ph, "= post_norm", [lambda s: lib.logismos_launch_post_norm(P(y), 1, P(None), m, P(x), P(ones), P(ones), P(h), 0, m, H, H, 1e-6, P(None), s)] * 4, 18.0 * m * H)
        cu1, sl, ps = ints(np.arange(m + 1)), ints(range(m)), ints([ctx - 1] * m)
        sz = 4.0 * m * gh * gk * gv
        ss, pr, low, w2, go = [zf(m, gh, gk, gv) for _ in range(copies(sz))], bf(m, g_main), rf(m, 32), bf(kw, 64), bf(m, vw)
        da = [gla_args(pr, None, low, w2, q, m, sl, cu1, go, 1) for q in ss]
        add(ph, "gated linear attention (with decay projection)", [lambda s, a=a: lib.logismos_launch_time_mix_step(Y(a), m, 0, s) for a in da], 2 * sz + m * (4.0 * kw + 6.0 * vw) + 2.0 * kw * RANK, like="time_mix_step")
        tz = 4.0 * m * kz["th"] * kz["td"] ** 2
        ss, rk, rl, rw, ro = [zf(m, kz["th"], kz["td"], kz["td"]) for _ in range(copies(tz))], bf(m, 4 * tdw), rf(m, kz["rank"]), bf(tdw, 2 * kz["rank"]), bf(m, tdw)
        db = [gla_args(rk, None, rl, rw, q, m, sl, cu1, ro, 0) for q in ss]
        add(ph, "= time_mix_step (with decay projection)", [lambda s, a=a: lib.logismos_launch_time_mix_step(Y(a), m, 0, s) for a in db], 2 * tz + m * tdw * 10.0 + 2.0 * tdw * kz["rank"])
        del ss
        nb = ctx // 16 + 1
        cl = torch.full((m,), ctx, dtype=torch.int32)
        tab, cg = ints(np.random.default_rng(1).permutation(m * nb).reshape(m, nb)), cl.to(dev)
        kp, vpool, dq, do, gd = bf(m * nb, 16, KD), bf(m * nb, 16, KD), bf(m, 2 * HD + 2 * KD), bf(m, HD), rf(m, hg)
        s1 = torch.randperm(m * nb * 16, device=dev)[:m].contiguous()
        add(ph, "q, k norm + rotation + store", [lambda s: lib.logismos_launch_qk_norm_rotary_store(P(dq), dq.shape[1], P(kp), P(vpool), P(s1), P(ps), m, heads, kv, DIM, DIM, P(ones), P(ones), 1e-6, P(table), 64,
                                                                                                   m * nb * 16, 0, P(st), s)] * 4, m * (4.0 * HD + 8.0 * KD), like="unit_qk_store")
        add(ph, "= unit_qk_store", [lambda s: lib.logismos_launch_unit_qk_store(P(dq), dq.shape[1], P(kp), P(vpool), P(s1), P(ps), m, heads, kv, DIM, DIM, 1e-6, 0.1, 1024.0, m * nb * 16, 0, P(st), s)] * 4,
            m * (4.0 * HD + 8.0 * KD))
        # windows rotate over shifted tables, so that the keys seen exceed L2 together
        vc = torch.full((m,), lib.logismos_window_context(ctx, WINDOW, KEEP), dtype=torch.int32)
        chunk = ops.pick_decode_chunk(vc, kv, DIM)
        while chunk <= 512 and chunk > 64 and -(-int(vc[0]) // chunk) * m * kv < 256:
            chunk //= 2
        offs, total = ops.build_decode_chunks(vc, chunk)
        offs = offs.to(dev)
        scr = torch.empty(max(16, lib.logismos_paged_decode_scratch_bytes(total, heads, DIM)), dtype=torch.uint8, device=dev)
        w = Window(DIM ** -0.5, WINDOW, KEEP, 1, A(gd), hg)
        tabw = [torch.roll(tab, 33 * i, 1).contiguous() for i in range(12)]
        add(ph, "window attention + merge (ctx %d)" % ctx, [lambda s, t=t: lib.logismos_launch_window_attention_decode_bf16(P(dq), dq.shape[1], P(kp), P(vpool), P(t), P(cg), P(offs), P(do), HD, P(scr), m, total, chunk,
                                                                                                                          nb, m * nb, heads, kv, DIM, Y(w), P(st), s) for t in tabw],
            m * (WINDOW + KEEP) * KD * 4.0, 4.0 * m * (WINDOW + KEEP) * HD, "biased decode at the window's length")
        cw = torch.full((m,), WINDOW + KEEP, dtype=torch.int32)
        pc = ops.pick_decode_chunk(cw, kv, DIM)
        o2, t2 = ops.build_decode_chunks(cw, pc)
        o2, cw = o2.to(dev), cw.to(dev)
        scr2 = torch.empty(max(16, lib.logismos_paged_decode_scratch_bytes(t2, heads, DIM)), dtype=torch.uint8, device=dev)
        b1 = ScoreBias(DIM ** -0.5, 30.0, A(tb), 1024, 5.0, 1.2 * DIM, A(dq) + (HD + 2 * KD) * 2, dq.shape[1], 1.0)
        add(ph, "= biased decode at the window's length", [lambda s, t=t: lib.logismos_launch_bias_attention_decode_bf16(P(dq), dq.shape[1], P(kp), P(vpool), P(t), P(cw), P(o2), P(do), HD, P(scr2), m, t2, pc, nb, m * nb,
                                                                                                                       heads, kv, DIM, Y(b1), P(st), s) for t in tabw], m * (WINDOW + KEEP) * KD * 4.0)
        del kp, vpool
        # latent attention
        raw = rf(m, NL)
        lr = LatentRotary(A(table), A(ps), R, ROT, A(gd), heads, hg)
        lpool, cqm = bf(m * nb, 16, Rp), bf(m, Q)
        add(ph, "latent norms + rotation + store", [lambda s: lib.logismos_launch_latent_norm_store(P(raw), NL, P(ones), P(ones), P(cqm), P(lpool), P(s1), m, Q, Q, Rp, R, 1e-6, m * nb * 16, 0, 1, Y(lr), P(st), s)] * 4,
            m * (10.0 * (Q + R + ROT) + 12.0 * heads), like="latent_norm_store")
        lp2 = bf(m * nb, 16, R)
        add(ph, "= latent_norm_store", [lambda s: lib.logismos_launch_latent_norm_store(P(raw), NL, P(ones), P(ones), P(cqm), P(lp2), P(s1), m, Q, Q, R, R, 1e-6, m * nb * 16, 0, 1, None, P(st), s)] * 4, m * 10.0 * (Q + R))
        qd, ql, ol = bf(m, HD), bf(m, heads * Rp), bf(m, heads * Rp)
        for rr, name, like in ((Rp, "", "latent decoder"), (R, "= ", None)):
            wk = [bf(heads, rr, DIM) for _ in range(copies(2.0 * heads * rr * DIM))]
            tagged = lambda n: name + n + (" (latent decoder)" if name else "")
            add(ph, tagged("latent queries per head"), [lambda s, w_=w_: lib.logismos_launch_linear_small_bf16(P(qd), P(w_), P(None), P(ql), m, rr, DIM, HD, heads * rr, heads, DIM, rr * DIM, rr, 0, 0.0, 0.0, 0.0, s) for w_ in wk],
                2.0 * heads * rr * DIM + 2.0 * m * (HD + heads * rr), 2.0 * m * heads * rr * DIM, like and "latent queries per head (latent decoder)")
            wv = [w_.view(heads, DIM, rr) for w_ in wk]
            add(ph, tagged("latent values per head"), [lambda s, w_=w_: lib.logismos_launch_linear_small_bf16(P(ol), P(w_), P(None), P(do), m, DIM, rr, heads * rr, HD, heads, rr, rr * DIM, DIM, 0, 0.0, 0.0, 0.0, s) for w_ in wv],
                2.0 * heads * rr * DIM + 2.0 * m * (HD + heads * rr), 2.0 * m * heads * rr * DIM, like and "latent values per head (latent decoder)")
            hl = cl.numpy()
            ck = lib.logismos_pick_latent_chunk(hl.ctypes.data_as(C.c_void_p), m, heads)
            lo, lt = ops.build_decode_chunks(cl, ck)
            lo = lo.to(dev)
            lscr = torch.empty(lib.logismos_latent_decode_scratch_bytes(lt, heads, rr), dtype=torch.uint8, device=dev)
            used = R + ROT if rr == Rp else R
            pl, g = (lpool, gd) if rr == Rp else (lp2, None)
            add(ph, tagged("latent decode + merge (ctx %d)" % ctx), [lambda s: lib.logismos_launch_latent_decode_bf16(P(ql), P(pl), P(tab), P(cg), P(lo), P(ol), P(lscr), m, lt, ck, nb, m * nb, heads, rr, 0.05, P(g), hg, P(table if rr == Rp else None), R, ROT, P(st), s)] * 3,
                2.0 * m * ctx * used, 2.0 * m * ctx * heads * (used + R), like and "latent decode + merge (latent decoder)")
        del lpool, lp2
    return rows
