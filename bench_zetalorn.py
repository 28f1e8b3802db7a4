"""Prefill and decode throughput of the Zetalorn decoder (pooled-window attention beside linear attention, and differential
attention over chunks, in turn, each with a mixture of experts) at sizes that resemble real layers, beside the Vugedra decoder,
whose executor, mixtures and bf16 weights it shares, at equal width, depth and attention heads (`bench.py --workload zetalorn`).

Random weights, bf16. Contexts are built by real chunked prefill steps through the same executor. A step's device work is
replayed and timed with CUDA events; the host-buffer entry point is timed around the same step. Every layer's weights, the
states and the cache of all contexts exceed L2 together."""
from __future__ import annotations

import ctypes as C

import numpy as np

import bench_vugedra as BV
from bench_latent import VOCAB, _graph_us

WINDOW, POOL, CHUNK, EXPERTS, TOP, GROUPS, KEEP = 512, 8, 1024, 16, 3, 4, 2
# width, layers; heads of both kinds of attention (kv: key heads), left ones of 128, differential ones of two maps of 64 over values of
# 128; linear-attention heads of lk x lv; expert size. A token uses as many experts as in the Vugedra decoder, the shared one included.
SIZES = {
    "1024x16": dict(width=1024, layers=16, heads=8, kv=2, lh=8, lk=64, lv=128, ff=512),
    "2048x16": dict(width=2048, layers=16, heads=16, kv=4, lh=16, lk=64, lv=128, ff=1024),
    "4096x8": dict(width=4096, layers=8, heads=32, kv=8, lh=32, lk=64, lv=128, ff=2048),
}
DIM, MAP = 128, 64
ROT, LIMIT = 64, 7.0


def is_pair(i):
    return i % 2 == 0


def zetalorn_config(z, vocab=VOCAB):
    moe = {"ff": z["ff"], "ff_kind": 2, "experts": EXPERTS, "top": TOP, "scoring": 1, "no_correction": 1, "route_groups": GROUPS, "keep_groups": KEEP, "glu_alpha": 1.702, "glu_limit": LIMIT,
           "glu_shift": 1.0}
    heads = {"heads": z["heads"], "kv_heads": z["kv"], "rot_dims": ROT, "rot_base": 1e4}
    pair = {"kind": 6, **heads, "dim": DIM, "vdim": DIM, "scale": DIM ** -0.5, "rot_halves": 1, "window": WINDOW, "pool": POOL, "lin_heads": z["lh"], "lin_dim": z["lk"], "lin_vdim": z["lv"],
            "decay": [1.0 - 2.0 ** (-1 - 8.0 * h / z["lh"]) for h in range(z["lh"])]}
    diff = {"kind": 5, **heads, "dim": MAP, "vdim": DIM, "scale": MAP ** -0.5, "window": CHUNK, "chunked": 1, "diff": 0.3, "rot_factor": 8.0}
    return {"vocab": vocab, "hidden": z["width"], "n_layers": z["layers"], "norm_eps": 1e-6, "norm": 2, "logit_scale": 1.0,
            "layers": [dict(pair if is_pair(i) else diff, **moe, weights_of=i) for i in range(z["layers"])]}


def zetalorn_weights(cfg, z, seed):
    """Layers of one kind, and experts, share their host arrays (every one still has its own copy on the device)."""
    rng = np.random.Generator(np.random.PCG64(seed))

    def bits(a):
        return (np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype(np.uint16)

    def mat(n, k, gain=1.0):
        return bits(rng.standard_normal((n, k), dtype=np.float32) * np.float32(gain / np.sqrt(k)))

    H, F, HD, KD, lk, lv = cfg["hidden"], z["ff"], z["heads"] * DIM, z["kv"] * DIM, z["lh"] * z["lk"], z["lh"] * z["lv"]
    ones, zeros = lambda n: bits(np.ones(n)), lambda n: bits(np.zeros(n))
    up, down, gate = mat(F, H), mat(H, F), mat(H, H)
    common = dict(norm1=ones(1), norm2=ones(1), rg1=gate, rg1_b=zeros(H), rg2=gate, rg2_b=zeros(H), router=mat(EXPERTS, H), experts=[up, up, down] * EXPERTS)
    q, k, o = mat(HD, H), mat(KD, H), mat(H, HD)
    pair = dict(common, left_q=q, left_k=k, left_v=k, left_q_norm=ones(DIM), left_k_norm=ones(DIM), left_o=o, left_out=ones(H), right_q=mat(lk, H), right_k=mat(lk, H), right_v=mat(lv, H),
                right_g=mat(lv, H), right_norm=ones(lv), right_o=mat(H, lv), right_out=ones(H))
    lam = bits(np.full(MAP, 0.1))
    diff = dict(common, q=q, k=k, v=k, q_norm=ones(MAP), k_norm=ones(MAP), lq1=lam, lk1=lam, lq2=lam, lk2=bits(np.full(MAP, 0.05)), o=o)
    return {"embed": mat(cfg["vocab"], H, np.sqrt(H)), "head": mat(cfg["vocab"], H), "final_norm": ones(1), "layers": [pair if is_pair(i) else diff for i in range(cfg["n_layers"])]}


class Engine(BV.Engine):
    def make(self, which, z, pool, mb, step_tokens, seqs, device, seed):
        if which != "zetalorn":
            return super().make(which, z, pool, mb, step_tokens, seqs, device, seed)
        from logismos_b200.zetalorn import ZetalornModel
        cfg = zetalorn_config(z)
        return cfg, ZetalornModel(cfg, zetalorn_weights(cfg, z, seed), pool, mb, step_tokens, seqs, seqs, device=device)


def mixer_params(z, pair):
    H, HD, KD = z["width"], z["heads"] * DIM, z["kv"] * DIM
    return H * (2 * HD + 2 * KD + H) + (H * z["lh"] * (2 * z["lk"] + 3 * z["lv"]) if pair else 0)


def stack_params(z, experts):
    """Matrix weights of all layers with so many experts each."""
    return sum(mixer_params(z, is_pair(i)) + 3 * z["width"] * z["ff"] * experts + z["width"] * (EXPERTS + z["width"]) for i in range(z["layers"]))


def active_experts(tokens):
    return EXPERTS * (1.0 - (1.0 - TOP / EXPERTS) ** tokens)


def seen_keys(z, pair, ctx):
    return min(ctx, WINDOW) + max(0, ctx - WINDOW) // POOL if pair else (ctx - 1) % CHUNK + 1


def decode_bytes(z, seqs, ctx, vocab=VOCAB):
    """Algorithmic HBM bytes of one decode step: weights of what is used once, cached rows that are seen, states."""
    by = 2.0 * (stack_params(z, active_experts(seqs)) + vocab * z["width"])
    for i in range(z["layers"]):
        by += seqs * (4.0 * seen_keys(z, is_pair(i), ctx + 1) * z["kv"] * DIM + (8.0 * z["lh"] * z["lk"] * z["lv"] if is_pair(i) else 0.0))
    return by


def attention_pairs(n, pair):
    """Query-key pairs of a prompt of n tokens."""
    i = np.arange(n)
    if pair:
        return float((np.minimum(i + 1, WINDOW) + np.maximum(i - WINDOW + 1, 0) // POOL).sum())
    return float((i % CHUNK + 1).sum())


def prefill_flops(z, seqs, n):
    fl = 2.0 * seqs * n * stack_params(z, TOP)
    for i in range(z["layers"]):
        # a map of a differential head: scores over 64 channels, values over 128, twice
        fl += (4.0 * DIM if is_pair(i) else 4.0 * (MAP + DIM)) * z["heads"] * seqs * attention_pairs(n, is_pair(i))
    return fl


def measure(sizes, iters, peaks, seqs=(8, 64), ctx=2048, prefill=(4, 1024)):
    import torch
    out = []
    for name in sizes:
        z, vz = SIZES[name], BV.SIZES[name]
        row = {"size": name, **z}
        for which in ("zetalorn", "vugedra"):
            own = which == "zetalorn"
            zz, M = (z, None) if own else (vz, BV)
            r = {"params": stack_params(z, EXPERTS) if own else BV.stack_params(vz, BV.EXPERTS), "params_per_token": stack_params(z, TOP) if own else BV.stack_params(vz, BV.active_experts())}
            e = Engine(which, zz, prefill[0], prefill[1], prefill[0] * prefill[1])
            e.step(list(range(prefill[0])), [0] * prefill[0], [prefill[1]] * prefill[0])
            ms, host = e.time(iters)
            T, fl = prefill[0] * prefill[1], prefill_flops(z, *prefill) if own else BV.prefill_flops(vz, *prefill)
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
                by = decode_bytes(z, n, ctx) if own else BV.decode_bytes(vz, n, ctx)
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
    """Every kernel of the Zetalorn decoder at one size, and the like kernels ("= ...") of the other decoders of the executor, each
    against its roofline (the slower of bytes over the measured copy bandwidth and FLOPs over the measured bf16 peak). Operands
    rotate over copies that exceed L2 together."""
    import torch
    from logismos_b200 import ops
    from logismos_b200._lib import check, i32, lib
    from logismos_b200.structs import GatedResidual, Groups, HeadNorm, MixtureOut, MoeRoute, Ssd, TanhNorm, TimeMix, Window
    dev, rows, keep = "cuda", [], []
    P = lambda t: C.c_void_p(t.data_ptr() if t is not None else 0)
    A = lambda t: 0 if t is None else t.data_ptr()
    Y = lambda n: C.byref(n)
    st = torch.zeros(1, dtype=torch.int32, device=dev)
    H, F, heads, kv, HD, KD = z["width"], z["ff"], z["heads"], z["kv"], z["heads"] * DIM, z["kv"] * DIM
    lh, lk, lv = z["lh"], z["lk"], z["lv"]
    kw, vw = lh * lk, lh * lv
    up = lambda v, m: (v + m - 1) // m * m
    bf = lambda *s: torch.randn(s, device=dev, dtype=torch.bfloat16) * 0.1
    rf = lambda *s: torch.randn(s, device=dev)
    zf = lambda *s: torch.zeros(s, device=dev)
    ints = lambda a: torch.as_tensor(np.asarray(a, np.int32)).to(dev)
    it = lambda *s: torch.zeros(s, dtype=torch.int32, device=dev)
    u8 = lambda n: torch.zeros(n, dtype=torch.uint8, device=dev)
    copies = lambda nbytes: max(2, min(12, int(3e8 // max(nbytes, 1)) + 1))
    streams = lambda m, n, k: m <= (16 if n * k >= 1 << 23 else 32)

    def add(phase, name, calls, nbytes, flops=0.0, like=None):
        us = _graph_us(calls)
        if int(st.item()):
            raise RuntimeError("%s / %s: device status 0x%x" % (phase, name, int(st.item())))
        roof = max(nbytes / peaks["hbm"] / 1e3, flops / peaks["tf_burst"] / 1e6)
        rows.append({"phase": phase, "kernel": name, "us": us, "roofline_us": roof, "frac": roof / us,
                     "bound": "hbm" if nbytes / peaks["hbm"] / 1e3 >= flops / peaks["tf_burst"] / 1e6 else "tensor", "like": like})

    def gemm(phase, name, m, n, k, epi, like=None):
        """A projection by the route that the executor takes for m rows."""
        ws, a = [bf(n, k) for _ in range(copies(2.0 * n * k))], bf(m, k)
        out = torch.zeros((m, n // 2 if epi == 2 else n), device=dev, dtype=torch.float32 if epi in (1, 3) else torch.bfloat16)
        if epi != 1 and streams(m, n, k):
            calls = [lambda s, w=w: lib.logismos_launch_linear_small_bf16(P(a), P(w), P(None), P(out), m, n, k, k, out.shape[1], 1, 0, 0, 0, epi, 0, 0, 0, s) for w in ws]
        else:
            calls = [lambda s, w=w: lib.logismos_launch_linear_t_act_bf16(P(a), P(w), P(None), P(out), m, n, k, k, out.shape[1], epi | 0x100, 0, 0, 0, P(st), s) for w in ws]
        add(phase, name, calls, 2.0 * n * k + 2.0 * m * k + out.numel() * out.element_size() * (2 if epi == 1 else 1), 2.0 * m * n * k, like)

    def grouped(phase, name, m, n_main, n_tail=0, silu=(0, 0), like=None):
        n = n_main + n_tail
        ws, a = [bf(n, H) for _ in range(copies(2.0 * n * H))], bf(m, H)
        out, tail, bias = torch.zeros((m, n_main), device=dev, dtype=torch.bfloat16), zf(m, max(n_tail, 1)), zf(n_main)
        g = Groups(1, (i32 * 8)(n), n_main, A(tail), n_tail, 0.0, 0, A(bias), *silu)
        keep.append((g, tail, bias))
        nbytes, flops = 2.0 * n * H + 2.0 * m * H + 2.0 * m * n_main + 4.0 * m * n_tail, 2.0 * m * n * H
        if 32 < m <= 512 and up(n, 128) // 128 * (up(m, 128) // 128) <= 74:   # summed over slices of k, then finished
            acc = zf(m, n)
            both = lambda s, w: lib.logismos_launch_linear_t_act_bf16(P(a), P(w), P(None), P(acc), m, n, H, H, n, 0x101, 0, 0, 0, P(st), s) or lib.logismos_launch_linear_groups_finish(P(acc), P(out), m, n, n, n_main, Y(g), s)
            return add(phase, name + " (with finish)", [lambda s, w=w: both(s, w) for w in ws], nbytes, flops, like)
        if streams(m, n, H):
            calls = [lambda s, w=w: lib.logismos_launch_linear_groups_small_bf16(P(a), P(w), P(out), m, n, H, H, n_main, Y(g), s) for w in ws]
        else:
            calls = [lambda s, w=w: lib.logismos_launch_linear_groups_tc_bf16(P(a), P(w), P(out), m, n, H, H, n_main, Y(g), P(st), s) for w in ws]
        add(phase, name, calls, nbytes, flops, like)

    ones, table = torch.ones(max(H, HD, vw), device=dev), rf(ctx + 16, 64)
    norm = TanhNorm(0.7, A(ones), A(ones))
    pair_n, diff_n = HD + 2 * KD + 2 * kw + 2 * vw + H, HD + 2 * KD + H
    silu = (HD + 2 * KD, HD + 2 * KD + 2 * kw + vw)
    vug_n = up(HD + 2 * KD, 128)

    def residuals(ph, m, zero):
        """The launches between sublayers: one branch, two, a mixture."""
        x, h, gate = rf(m, H), bf(m, H), bf(m, H)
        sets = [(rf(m, H), rf(m, H)) for _ in range(copies(8.0 * m * H))]

        def args(b, mix=None):
            r = GatedResidual(x=A(x), zero_branches=zero, gate=A(gate), ld_gate=H, h=A(h), gain=1.0, eps=1e-6, n_src_rows=m, rows=m, n=H, ld=H)
            r.branch[0] = A(b[0]) if b else 0
            if b and len(b) > 1:
                r.branch[1], r.branch_gain[0], r.branch_gain[1] = A(b[1]), A(ones), A(ones)
            if mix is not None:
                r.mixture = C.pointer(mix)
            keep.append((r, mix, x, h, gate))
            return r
        one, two = [args(b[:1]) for b in sets], [args(b) for b in sets]
        z4 = 4.0 * zero
        add(ph, "gated residual + norm", [lambda s, r=r: lib.logismos_launch_gated_residual(Y(r), P(st), s) for r in one], m * H * (16.0 + z4), like="post_norm")
        add(ph, "norms of both branches + gated residual + norm", [lambda s, r=r: lib.logismos_launch_gated_residual(Y(r), P(st), s) for r in two], m * H * (20.0 + 2 * z4), like="post_norm")
        add(ph, "= post_norm", [lambda s, b=b: lib.logismos_launch_post_norm(P(b[0]), zero, P(None), m, P(x), P(ones), P(ones), P(h), 0, m, H, H, 1e-6, P(None), s) for b in sets], m * H * (14.0 + z4))
        return args

    def mixture(ph, m, args):
        few = lib.logismos_moe_streams(m, TOP, EXPERTS, 0, 0, H, F)
        ld = up(EXPERTS, 16)
        logits, h, corr = rf(m, ld), bf(m, H), zf(ld)
        wts, prow, ident, off, tok = zf(m, TOP), it(m, TOP), zf(m), it(EXPERTS + 1), it(m * TOP)
        counts, pe = it(EXPERTS), it(m, TOP)
        mt = lib.logismos_moe_max_tiles(m, TOP, EXPERTS, 0)
        tiles, nt, gat = it(mt, 4), it(1), bf(m * TOP, H)

        def route(own):
            r = MoeRoute(A(logits), ld, 0, 0 if own else A(corr), EXPERTS, 0, TOP, 0, A(wts), A(prow), A(ident))
            if own:
                r.scoring, r.groups, r.keep_groups = 1, GROUPS, KEEP
            if few:
                r.offsets, r.row_token = A(off), A(tok)
            else:
                r.counts, r.pair_expert, r.tiles, r.n_tiles = A(counts), A(pe), A(tiles), A(nt)
            return r
        r, soft = route(True), route(False)
        keep.append((r, soft, logits, corr, wts, prow, ident, off, tok, counts, pe, tiles, nt))

        def choose(s, r=r):
            if not few:
                counts.zero_()
            return lib.logismos_launch_moe_route(Y(r), m, s)
        name = "choice of experts" + ("" if few else " (with clearing)")
        add(ph, "= %s, softmax" % name, [lambda s: choose(s, soft)] * 4, m * (ld * 4.0 + 12.0 * TOP))
        add(ph, name, [choose] * 4, m * (ld * 4.0 + 12.0 * TOP), like="%s, softmax" % name)
        check(choose(torch.cuda.current_stream().cuda_stream), "moe_route")
        rows_of = (off[1:] - off[:-1] if few else counts).cpu().numpy()
        n_rows, used = int(rows_of.sum()), int((rows_of > 0).sum())
        nw = max(2, min(6, int(3e8 // (6.0 * F * H * EXPERTS)) + 1))
        wu, wd = [bf(EXPERTS, 2 * F, H) for _ in range(nw)], [bf(EXPERTS, H, F) for _ in range(nw)]
        mid, out = bf(m * TOP, F), bf(m * TOP, H)
        ub, ul = 2.0 * used * 2 * F * H + 2.0 * m * H + 2.0 * n_rows * F, 4.0 * n_rows * F * H
        db, dl = 2.0 * used * F * H + 2.0 * n_rows * F + 2.0 * n_rows * H, 2.0 * n_rows * F * H
        if few:
            ex = 8 if m <= 8 else 16
            call = lambda s, w, epi: lib.logismos_launch_linear_experts_small_bf16(P(h), P(w), P(mid), P(off), P(tok), EXPERTS, m, ex, 2 * F, H, H, F, epi, 1.702, LIMIT, 1.0, s)
            down = lambda s, w: lib.logismos_launch_linear_experts_small_bf16(P(mid), P(w), P(out), P(off), P(None), EXPERTS, m, ex, H, F, F, H, 0, 0, 0, 0, s)
        else:
            add(ph, "rows by expert", [lambda s: lib.logismos_launch_moe_place(Y(r), P(h), P(gat), H, m, s)] * 4, 2.0 * H * (m + n_rows), like="the same kernel")
            call = lambda s, w, epi: lib.logismos_launch_linear_experts_tc_bf16(P(gat), m * TOP, P(None), 0, P(w), P(mid), P(tiles), P(nt), mt, EXPERTS, 2 * F, H, H, F, epi, 1.702, LIMIT, 1.0, P(st), s)
            down = lambda s, w: lib.logismos_launch_linear_experts_tc_bf16(P(mid), m * TOP, P(None), 0, P(w), P(out), P(tiles), P(nt), mt, EXPERTS, H, F, F, H, 0, 0, 0, 0, P(st), s)
        add(ph, "experts, gate and up (clamped)", [lambda s, w=w: call(s, w, 4) for w in wu], ub, ul, "experts, gate and up (silu)")
        add(ph, "= experts, gate and up (silu)", [lambda s, w=w: call(s, w, 2) for w in wu], ub, ul)
        add(ph, "experts, down", [lambda s, w=w: down(s, w) for w in wd], db, dl, "the same kernel")
        del wu, wd
        outs = [bf(m * TOP, H) for _ in range(copies(2.0 * m * TOP * H))]
        mo = [MixtureOut(A(o), A(prow), A(wts), A(ident), TOP, TOP, 0, 0) for o in outs]
        keep.append((outs, mo))
        rs, x = [args(None, o) for o in mo], rf(m, H)
        add(ph, "sum of the experts + gated residual + norm", [lambda s, r=r: lib.logismos_launch_gated_residual(Y(r), P(st), s) for r in rs], m * H * 12.0 + 2.0 * n_rows * H, like="sum of the experts + tanh norms")
        add(ph, "= sum of the experts + tanh norms", [lambda s, o=o: lib.logismos_launch_tanh_norm(P(None), 0, Y(o), P(None), m, P(x), Y(norm), P(h), Y(norm), 0, m, H, P(st), s) for o in mo], m * H * 10.0 + 2.0 * n_rows * H)

    decay = 1.0 - 2.0 ** (-1.0 - 8.0 * torch.arange(lh, device=dev) / lh)
    decay = torch.stack([torch.log2(decay), decay, torch.zeros_like(decay)], dim=1).float().contiguous()

    def linear_args(proj, state, slots, cu, y):
        fresh = u8(slots.numel())
        keep.append(fresh)
        return Ssd(state=A(state), state_slots=A(slots), fresh=A(fresh), cu=A(cu), y=A(y), ld_y=vw, heads=lh, groups=lh, np=lk, vp=lv, xbc=A(proj), ld_xbc=proj.shape[1], decay=A(decay))

    def gla_args(proj, zz, low, w2, state, slots, cu, out):
        q = [torch.full((kw,), 2.0, device=dev), u8(slots.numel())]
        keep.append(q)
        return TimeMix(A(proj), proj.shape[1], 0, kw, 2 * kw, 2 * kw + vw, A(zz), kw, A(low), 32, A(w2), 64, 32, A(q[0]), 0, A(ones), A(state), A(slots), A(q[1]), A(cu), A(out), vw, lh, lv, lk,
                       1.0, 1e-6, 1, lv, 16.0, lk ** -0.5)

    def head_args(qkv, m, maps, pools, means, tabs, seqs, slots, pos, nb, qx):
        r = HeadNorm(qkv=A(qkv), ld=qkv.shape[1], rows=m, heads=heads, n_kv=kv, maps=maps, hd=DIM // maps, dim=DIM // maps, gain_q=A(ones), gain_k=A(ones), eps=1e-6, table=A(table), rot_dims=ROT,
                     q_out=A(qx), ld_q=2 * HD, k_pool=A(pools[0]), v_pool=A(pools[1]), slots=A(slots), positions=A(pos), n_pool_slots=nb * 16)
        if means:
            r.pool, r.pool_rows, r.k_mean, r.v_mean, r.tables, r.seq_ids, r.max_blocks, r.n_pool_blocks = POOL, (m if m <= 512 else 0), A(means[0]), A(means[1]), A(tabs), A(seqs), tabs.shape[1], nb
        keep.append(r)
        return r

    # ---- prefill of T tokens in sequences of 1024
    ph, nq = "prefill", T // 1024
    cu, slots, pos, seq_ids = ints(np.arange(nq + 1) * 1024), ints(range(nq)), ints(np.tile(np.arange(1024), nq)), ints(np.repeat(np.arange(nq), 1024))
    args = residuals(ph, T, 0)
    grouped(ph, "projections, pair", T, pair_n, silu=silu, like="projections, attention")
    grouped(ph, "projections, differential", T, diff_n, like="projections, attention")
    grouped(ph, "= projections, attention", T, vug_n, 16)
    nblk = 1024 // 16
    nb = nq * nblk
    perm = np.random.default_rng(0).permutation(nb).reshape(nq, nblk)
    tabs, kv_lens = ints(perm), ints([1024] * nq)
    slot64 = torch.as_tensor((perm[:, :, None] * 16 + np.arange(16)).reshape(-1).astype(np.int64)).to(dev)
    pools, means = (bf(nb, 16, KD), bf(nb, 16, KD)), (bf(nb, 2, KD), bf(nb, 2, KD))
    qkvs = [bf(T, HD + 2 * KD) for _ in range(copies(2 * T * (HD + 2 * KD)))]
    att, qx = bf(T, HD), bf(T, 2 * HD)
    ha = [head_args(q, T, 1, pools, means, tabs, seq_ids, slot64, pos, nb, None) for q in qkvs]
    hb = [head_args(q, T, 2, pools, None, tabs, seq_ids, slot64, pos, nb, qx) for q in qkvs]
    move = T * (4.0 * HD + 8.0 * KD)
    add(ph, "q, k norm + rotation + store, pair", [lambda s, a=a: lib.logismos_launch_head_norm_store(Y(a), 0, P(st), s) for a in ha], move, like="q, k norm + rotation + store, whole rows")
    add(ph, "q, k norm + rotation + store, differential", [lambda s, a=a: lib.logismos_launch_head_norm_store(Y(a), 0, P(st), s) for a in hb], T * (6.0 * HD + 8.0 * KD), like="q, k norm + rotation + store, whole rows")
    add(ph, "= q, k norm + rotation + store, whole rows", [lambda s, q=q: lib.logismos_launch_qk_norm_rotary_store(P(q), q.shape[1], P(pools[0]), P(pools[1]), P(slot64), P(pos), T, heads, kv, DIM, DIM, P(ones), P(ones),
                                                                                                                  1e-6, P(table), ROT, T, 0, P(st), s) for q in qkvs], move)
    add(ph, "means of blocks", [lambda s: lib.logismos_launch_pool_blocks(Y(ha[0]), 0, P(st), s)] * 4, T * 4.0 * KD * (1 + 1 / POOL), like="q, k norm + rotation + store, whole rows")
    gate = rf(T, 2 * heads)
    wins = {"pooled": Window(scale=DIM ** -0.5, size=WINDOW, pool=POOL, k_mean=A(means[0]), v_mean=A(means[1])), "chunked": Window(scale=MAP ** -0.5, size=CHUNK, chunked=1),
            "kept": Window(DIM ** -0.5, WINDOW, 4, 1, A(gate), heads)}
    scr = torch.empty(lib.logismos_paged_prefix_attention_scratch_bytes(T * 2, nq, kv, DIM), dtype=torch.uint8, device=dev)

    def prefix(s, q, w, out, nh):
        n = lib.logismos_window_view_keys(Y(w), 1024, 1024)
        return lib.logismos_launch_window_attention_prefix_bf16(P(q), q.shape[1], P(cu), P(kv_lens), P(pools[0]), P(pools[1]), P(tabs), nblk, nb, P(out), nh * DIM, P(scr), T, n * nq, nq, 1024, n, nh, kv, DIM,
                                                                Y(w), P(st), s)
    kvb = T * 8.0 * KD
    add(ph, "pooled-window attention (with gather)", [lambda s, q=q: prefix(s, q, wins["pooled"], att, heads) for q in qkvs], T * 4.0 * HD + kvb, 4.0 * HD * nq * attention_pairs(1024, True), "window attention (with gather)")
    add(ph, "= window attention (with gather)", [lambda s, q=q: prefix(s, q, wins["kept"], att, heads) for q in qkvs], T * 4.0 * HD + kvb, 4.0 * HD * nq * BV.window_pairs(1024))

    def differential(s):
        n = lib.logismos_window_view_keys(Y(wins["chunked"]), 1024, 1024)
        return lib.logismos_launch_differential_prefix_bf16(P(qx), 2 * HD, P(cu), P(kv_lens), P(pools[0]), P(pools[1]), P(tabs), nblk, nb, P(att), HD, P(scr), T, n * nq, nq, 1024, n, heads, kv, DIM,
                                                            Y(wins["chunked"]), DIM, 0.4, 0.7, 1e-6, P(st), s)
    add(ph, "differential attention (with gather)", [differential] * 4, T * 4.0 * HD + kvb, 4.0 * heads * (MAP + DIM) * nq * attention_pairs(1024, False), "window attention (with gather)")
    del qkvs, qx
    prs, lst, ly = [bf(T, 2 * kw + 2 * vw) for _ in range(copies(4 * T * (kw + vw)))], zf(nq, lh, lk, lv), bf(T, vw)
    la = [linear_args(q, lst, slots, cu, ly) for q in prs]
    rec_b, rec_f = T * (4.0 * kw + 4.0 * vw), T * lh * (4.0 * lk * lv + 64.0 * (lk + lv))
    entries = lib.logismos_ssd_segments(T, nq, 1024, lh)
    seg = torch.empty(max(16, lib.logismos_ssd_scratch_bytes(entries, lh, lk, lv)), dtype=torch.uint8, device=dev)
    add(ph, "linear attention", [lambda s, a=a: lib.logismos_launch_ssd_segmented_bf16(Y(a), nq, 1024, P(seg), entries, s) for a in la], rec_b, rec_f, "gated linear attention")
    gq, zz, go = [bf(T, 2 * kw + 2 * vw) for _ in range(2)], rf(T, kw) + 2.0, bf(T, vw)
    ga = [gla_args(q, zz, None, None, lst, slots, cu, go) for q in gq]
    add(ph, "= gated linear attention", [lambda s, a=a: lib.logismos_launch_time_mix_chunked_bf16(Y(a), nq, s) for a in ga], T * (8.0 * kw + 6.0 * vw), T * lh * (4.0 * lk * lv + 32.0 * (lk + lv)))
    ys = [bf(T, vw) for _ in range(copies(2 * T * vw))]
    add(ph, "norm and gate of the linear attention", [lambda s, y=y: lib.logismos_launch_norm_gate(P(y), vw, P(prs[0]), prs[0].shape[1], P(ones), P(go), vw, 0, T, lh, lv, lv, 1e-6, s) for y in ys], 6.0 * T * vw,
        like="gate and norm of a state-space layer")
    add(ph, "= gate and norm of a state-space layer", [lambda s, y=y: lib.logismos_launch_gated_group_norm(P(y), vw, P(prs[0]), prs[0].shape[1], P(ones), P(go), vw, 0, T, lh, lv, lv, 1, 1e-6, s) for y in ys], 6.0 * T * vw)
    del prs, gq, ys
    gemm(ph, "output projection (left, differential)", T, H, HD, 3, like="the same kernel")
    gemm(ph, "output projection, right", T, H, vw, 3, like="the same kernel")
    grouped(ph, "gate and router", T, up(H, 128), up(EXPERTS, 16), like="projections, attention")
    mixture(ph, T, args)
    # ---- decode
    for m in batches:
        ph, acc = "decode %d" % m, 32 < m
        args = residuals(ph, m, 1)
        grouped(ph, "projections, pair", m, pair_n, silu=silu, like="projections, attention")
        grouped(ph, "projections, differential", m, diff_n, like="projections, attention")
        grouped(ph, "= projections, attention", m, vug_n, 16)
        if m <= 16:
            ws, a, yo = [bf(2, H, HD) for _ in range(copies(4.0 * H * HD))], bf(m, 2 * HD), rf(2, m, H)
            add(ph, "output projections, pair", [lambda s, w=w: lib.logismos_launch_linear_small_bf16(P(a), P(w), P(None), P(yo), m, H, HD, 2 * HD, H, 2, HD, H * HD, m * H, 3, 0, 0, 0, s) for w in ws],
                4.0 * H * HD + 4.0 * m * HD + 8.0 * m * H, 4.0 * m * H * HD, "the same kernel")
            del ws
        gemm(ph, "output projection (left, differential)", m, H, HD, 1 if m > 16 else 3, like="the same kernel")
        if m > 16:
            gemm(ph, "output projection, right", m, H, vw, 1, like="the same kernel")
        grouped(ph, "gate and router", m, up(H, 128), up(EXPERTS, 16), like="projections, attention")
        mixture(ph, m, args)
        cu1, sl, ps = ints(np.arange(m + 1)), ints(range(m)), ints([ctx - 1] * m)
        sz = 4.0 * m * lh * lk * lv
        ss, pr, low, w2, go = [zf(m, lh, lk, lv) for _ in range(copies(sz))], bf(m, 2 * kw + 2 * vw), rf(m, 32), bf(kw, 64), bf(m, vw)
        la = [linear_args(pr, q, sl, cu1, go) for q in ss]
        add(ph, "linear attention", [lambda s, a=a: lib.logismos_launch_ssd_step(Y(a), m, 0, s) for a in la], 2 * sz + m * (4.0 * kw + 4.0 * vw), like="gated linear attention (with decay projection)")
        ga = [gla_args(pr, None, low, w2, q, sl, cu1, go) for q in ss]
        add(ph, "= gated linear attention (with decay projection)", [lambda s, a=a: lib.logismos_launch_time_mix_step(Y(a), m, 0, s) for a in ga], 2 * sz + m * (4.0 * kw + 6.0 * vw) + 2.0 * kw * BV.RANK)
        add(ph, "norm and gate of the linear attention", [lambda s: lib.logismos_launch_norm_gate(P(go), vw, P(pr), pr.shape[1], P(ones), P(go), vw, 0, m, lh, lv, lv, 1e-6, s)] * 4, 6.0 * m * vw,
            like="gate and norm of a state-space layer")
        add(ph, "= gate and norm of a state-space layer", [lambda s: lib.logismos_launch_gated_group_norm(P(go), vw, P(pr), pr.shape[1], P(ones), P(go), vw, 0, m, lh, lv, lv, 1, 1e-6, s)] * 4, 6.0 * m * vw)
        del ss
        per = ctx // 16 + 1
        nb = m * per
        perm = np.random.default_rng(1).permutation(nb).reshape(m, per)
        tab, cg = ints(perm), ints([ctx] * m)
        pools, means, dq, do, qx, gd = (bf(nb, 16, KD), bf(nb, 16, KD)), (bf(nb, 2, KD), bf(nb, 2, KD)), bf(m, HD + 2 * KD), bf(m, HD), bf(m, 2 * HD), rf(m, heads)
        s1 = torch.as_tensor((perm[:, (ctx - 1) // 16] * 16 + (ctx - 1) % 16).astype(np.int64)).to(dev)
        ha, hb = head_args(dq, m, 1, pools, means, tab, ints(range(m)), s1, ps, nb, None), head_args(dq, m, 2, pools, None, tab, ints(range(m)), s1, ps, nb, qx)
        move = m * (4.0 * HD + 8.0 * KD)
        add(ph, "q, k norm + rotation + store, pair, at the end of a block", [lambda s: lib.logismos_launch_head_norm_store(Y(ha), 0, P(st), s)] * 4, move + m * 4.0 * KD * POOL, like="q, k norm + rotation + store, whole rows")
        add(ph, "q, k norm + rotation + store, differential", [lambda s: lib.logismos_launch_head_norm_store(Y(hb), 0, P(st), s)] * 4, m * (6.0 * HD + 8.0 * KD), like="q, k norm + rotation + store, whole rows")
        add(ph, "= q, k norm + rotation + store, whole rows", [lambda s: lib.logismos_launch_qk_norm_rotary_store(P(dq), dq.shape[1], P(pools[0]), P(pools[1]), P(s1), P(ps), m, heads, kv, DIM, DIM, P(ones), P(ones), 1e-6,
                                                                                                                 P(table), ROT, nb * 16, 0, P(st), s)] * 4, move)
        tabw = [torch.roll(tab, 33 * i, 1).contiguous() for i in range(12)]   # shifted tables, so that the keys seen exceed L2 together
        wins = {"pooled": Window(scale=DIM ** -0.5, size=WINDOW, pool=POOL, k_mean=A(means[0]), v_mean=A(means[1])), "chunked": Window(scale=MAP ** -0.5, size=CHUNK, chunked=1),
                "kept": Window(DIM ** -0.5, WINDOW, 4, 1, A(gd), heads)}

        def decode(name, w, q, out, nh, seen, like, differential=False):
            vc = torch.full((m,), lib.logismos_window_view_context(Y(w), ctx), dtype=torch.int32)
            chunk = ops.pick_decode_chunk(vc, kv, DIM)
            while chunk <= 512 and chunk > 64 and -(-int(vc[0]) // chunk) * m * kv < 256:
                chunk //= 2
            offs, total = ops.build_decode_chunks(vc, chunk)
            offs = offs.to(dev)
            scr = torch.empty(max(16, lib.logismos_paged_decode_scratch_bytes(total, 2 * nh, DIM)), dtype=torch.uint8, device=dev)
            launch, more = (lib.logismos_launch_differential_decode_bf16, (DIM, 0.4, 0.7, 1e-6)) if differential else (lib.logismos_launch_window_attention_decode_bf16, ())
            call = lambda s, t: launch(P(q), q.shape[1], P(pools[0]), P(pools[1]), P(t), P(cg), P(offs), P(out), nh * DIM, P(scr), m, total, chunk, per, nb, nh, kv, DIM, Y(w), *more, P(st), s)
            add(ph, "%s (ctx %d)" % (name, ctx), [lambda s, t=t: call(s, t) for t in tabw], m * seen * KD * 4.0, 0.0, like and "%s (ctx %d)" % (like, ctx))
        decode("pooled-window attention + merge", wins["pooled"], dq, do, heads, seen_keys(z, True, ctx), "window attention + merge")
        decode("= window attention + merge", wins["kept"], dq, do, heads, WINDOW + 4, None)
        decode("differential attention + merge with difference", wins["chunked"], qx, do, heads, CHUNK, "window attention + merge", True)
        gemm(ph, "head", m, VOCAB, H, 3, like="the same kernel")
        del pools, means
    return rows
