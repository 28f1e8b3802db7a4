"""The kernels of the Zetalorn decoder, each against the plain function of zetalorn_reference.py."""
import ctypes as C

import numpy as np
import pytest
import torch

import zetalorn_reference as R
from logismos_b200._lib import check, lib
from logismos_b200.structs import GatedResidual, Groups, HeadNorm, MixtureOut, MoeRoute, Ssd, Window

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
vp, i32 = C.c_void_p, C.c_int32
P = lambda t: vp(0 if t is None else t.data_ptr())
A = lambda t: 0 if t is None else t.data_ptr()
stream = lambda: vp(torch.cuda.current_stream().cuda_stream)


def dev(a, dtype):
    return torch.from_numpy(np.ascontiguousarray(a)).to(DEV).to(dtype)


fl = lambda a: dev(np.asarray(a, np.float32), torch.float32)
ints = lambda a: dev(np.asarray(a, np.int32), torch.int32)
host = lambda t: t.detach().float().cpu().numpy().astype(np.float64)
FP32 = pytest.mark.parametrize("fp32", [False, True])


def act(a, fp32):
    return fl(a) if fp32 else dev(np.asarray(a, np.float32), torch.bfloat16)


def close(got, want, tol):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    err = np.sqrt(np.mean((got - want) ** 2)) / np.sqrt(np.mean(want ** 2))
    assert err <= tol and np.abs(got - want).max() <= 12 * tol * np.abs(want).max(), (err, np.abs(got - want).max(), np.abs(want).max())


def status():
    return torch.zeros(1, dtype=torch.int32, device=DEV)


def padded(x, to):
    out = np.zeros(x.shape[:-1] + (to,))
    out[..., :x.shape[-1]] = x
    return out


def angles(rot, positions):
    a = np.arange(positions)[:, None] * R.rotary_frequencies(rot)
    return fl(np.stack([np.cos(a), np.sin(a)], axis=-1).reshape(positions, -1))


# ---- pages -----------------------------------------------------------------------------------------

class Cache:
    """Sequences with random keys and values in shuffled pages, and their pooled blocks."""

    def __init__(self, rng, lens, G, D, dim, vdim, fp32, pool=0, spare=3):
        self.G, self.D, self.lens, self.pool = G, D, lens, pool
        self.mb = max(-(-n // 16) for n in lens) + 1
        self.nb = sum(-(-n // 16) for n in lens) + spare
        perm, at = rng.permutation(self.nb), 0
        tables = -np.ones((len(lens), self.mb), np.int32)
        kp, v_ = (np.full((self.nb, 16, G * D), np.nan) for _ in range(2))     # what no sequence owns must not be touched
        rows = -(-16 // pool) if pool else 1
        km, vm = (np.full((self.nb, rows, G * D), np.nan) for _ in range(2))
        self.k, self.v, self.km, self.vm = [], [], [], []
        for s, n in enumerate(lens):
            b = -(-n // 16)
            tables[s, :b] = perm[at:at + b]
            at += b
            for store, means, pages, pooled, d in ((self.k, self.km, kp, km, dim), (self.v, self.vm, v_, vm, vdim)):
                x = host(act(padded(rng.standard_normal((n, G, d)), D), fp32))
                store.append(x)
                for t in range(n):
                    pages[tables[s, t // 16], t % 16] = x[t].reshape(-1)
                if pool:
                    m = host(act(R.pooled(x, pool), fp32)) if n >= pool else np.zeros((0, G, D))
                    means.append(m)
                    ends = [(i + 1) * pool - 1 for i in range(len(m))]
                    for i, e in enumerate(ends):
                        pooled[tables[s, e // 16], sum(f // 16 == e // 16 for f in ends[:i])] = m[i].reshape(-1)
        self.np_tables = tables
        self.tables, self.kp, self.vp, self.kmean, self.vmean = ints(tables), act(kp, fp32), act(v_, fp32), act(km, fp32), act(vm, fp32)

    def window(self, scale, size, chunked, out_f32=0):
        return Window(scale=scale, size=size, chunked=chunked, pool=self.pool, k_mean=A(self.kmean) if self.pool else 0, v_mean=A(self.vmean) if self.pool else 0, out_f32=out_f32)

    def want(self, s, rows, q, scale, size, chunked):
        """rows: positions; q [n, H, D] -> [n, H, D]."""
        n = self.lens[s]
        k, v, mask = self.k[s], self.v[s], (R.chunk_mask if chunked else R.window_mask)(n, size)
        if self.pool:
            k, v = np.concatenate([self.km[s], k]), np.concatenate([self.vm[s], v])
            mask = np.concatenate([R.pooled_mask(n, size, self.pool), mask], axis=1)
        return R.attend(q, k, v, scale, mask[rows])


VIEWS = [(1, 0, 1), (7, 0, 1), (64, 0, 1), (130, 0, 1), (1000, 0, 1), (1, 1, 0), (5, 3, 0), (16, 16, 0), (40, 8, 0), (130, 5, 0), (9, 40, 0), (128, 1, 0), (300, 7, 0), (33, 0, 0)]
SIZES = [(6, 2, 64, 20, 28), (20, 1, 64, 64, 64), (4, 4, 128, 100, 90), (2, 1, 256, 130, 200)]


def decode_call(c, qd, H, w, chunk, out, diff=None):
    n, G, D = len(c.lens), c.G, c.D
    vctx = np.array([lib.logismos_window_view_context(C.byref(w), v) for v in c.lens], np.int32)
    off = np.empty(n + 1, np.int32)
    total = lib.logismos_build_decode_chunks(vctx.ctypes.data_as(vp), n, chunk, off.ctypes.data_as(vp))
    scr = torch.full((max(1, lib.logismos_paged_decode_scratch_bytes(total, 2 * H, D)),), 255, dtype=torch.uint8, device=DEV)
    keep, st = [ints(c.lens), ints(off)], status()
    launch = lib.logismos_launch_differential_decode_bf16 if diff else lib.logismos_launch_window_attention_decode_bf16
    check(launch(P(qd), qd.shape[1], P(c.kp), P(c.vp), P(c.tables), P(keep[0]), P(keep[1]), P(out), out.shape[1], P(scr), n, total, chunk, c.mb, c.nb, H, G, D, C.byref(w), *(diff or ()),
                 P(st), stream()), "decode")
    torch.cuda.synchronize()
    assert st.item() == 0


@pytest.mark.parametrize("size,pool,chunked", VIEWS)
@pytest.mark.parametrize("H,G,D,dim,vdim", SIZES)
def test_decoded_tokens_see_their_window(H, G, D, dim, vdim, size, pool, chunked):
    rng = np.random.default_rng(size + pool)
    lens = [1, 2, 15, 16, 17, 33, 64, 65, 130, 145, 300, 700]
    c = Cache(rng, lens, G, D, dim, vdim, False, pool)
    n, scale = len(lens), 2.0 / np.sqrt(dim)
    qd = act(np.concatenate([padded(rng.standard_normal((n, H, dim)), D).reshape(n, -1), np.zeros((n, 16))], axis=1), False)
    q = host(qd)[:, :H * D].reshape(n, H, D)
    want = np.concatenate([c.want(s, [lens[s] - 1], q[s:s + 1], scale, size, chunked) for s in range(n)])
    for chunk, f32 in ((64, 0), (512, 1)):
        out = act(np.zeros((n, H * D + 8)), bool(f32))
        decode_call(c, qd, H, c.window(scale, size, chunked, f32), chunk, out)
        close(host(out)[:, :H * D].reshape(n, H, D), want, 6e-3)


@pytest.mark.parametrize("size,pool,chunked", VIEWS)
@pytest.mark.parametrize("H,G,D,dim,vdim", [SIZES[0], SIZES[2], SIZES[3]])
def test_prompts_see_their_windows(H, G, D, dim, vdim, size, pool, chunked):
    rng = np.random.default_rng(size + pool + 1)
    lens, new = [2, 130, 300, 700, 523, 411], [2, 130, 2, 300, 129, 17]
    c = Cache(rng, lens, G, D, dim, vdim, False, pool)
    T, n, scale = sum(new), len(lens), 2.0 / np.sqrt(dim)
    qd = act(padded(rng.standard_normal((T, H, dim)), D).reshape(T, -1), False)
    q, cu = host(qd).reshape(T, H, D), np.concatenate([[0], np.cumsum(new)]).astype(np.int32)
    rows = lambda s: np.arange(lens[s] - new[s], lens[s])
    want = np.concatenate([c.want(s, rows(s), q[cu[s]:cu[s + 1]], scale, size, chunked) for s in range(n)])
    for f32 in (0, 1):
        w, st = c.window(scale, size, chunked, f32), status()
        keys = [lib.logismos_window_view_keys(C.byref(w), a, b) for a, b in zip(lens, new)]
        scr = torch.empty(lib.logismos_paged_prefix_attention_scratch_bytes(sum(keys), n, G, D), dtype=torch.uint8, device=DEV)
        scr.fill_(255)
        out, keep = act(np.zeros((T, H * D + 8)), bool(f32)), [ints(cu), ints(lens)]
        check(lib.logismos_launch_window_attention_prefix_bf16(P(qd), H * D, P(keep[0]), P(keep[1]), P(c.kp), P(c.vp), P(c.tables), c.mb, c.nb, P(out), H * D + 8, P(scr), T, sum(keys), n, max(new),
                                                               max(keys), H, G, D, C.byref(w), P(st), stream()), "prefix")
        close(host(out)[:, :H * D].reshape(T, H, D), want, 6e-3)
        assert st.item() == 0


@pytest.mark.parametrize("size,pool,chunked", VIEWS)
def test_window_attention_in_fp32(size, pool, chunked):
    rng = np.random.default_rng(size + pool + 2)
    H, G, D, dim, vdim, lens = 6, 3, 64, 40, 50, [1, 65, 300]
    c = Cache(rng, lens, G, D, dim, vdim, True, pool)
    rows = [(s, p) for s, n in enumerate(lens) for p in sorted({0, n // 2, n - 1})]
    T = len(rows)
    qd = fl(padded(rng.standard_normal((T, H, dim)), D).reshape(T, -1))
    out, st, w, keep = fl(np.zeros((T, H * D))), status(), c.window(0.4, size, chunked), [ints([r[0] for r in rows]), ints([r[1] for r in rows])]
    check(lib.logismos_launch_window_attention_f32(P(qd), H * D, P(c.kp), P(c.vp), P(c.tables), P(keep[0]), P(keep[1]), P(out), H * D, T, c.mb, c.nb, H, G, D, C.byref(w), P(st), stream()), "f32")
    want = np.concatenate([c.want(s, [p], host(qd).reshape(T, H, D)[i:i + 1], 0.4, size, chunked) for i, (s, p) in enumerate(rows)])
    close(host(out).reshape(T, H, D), want, 3e-6)
    assert st.item() == 0


def test_a_page_that_is_missing_raises_the_status():
    rng = np.random.default_rng(0)
    c = Cache(rng, [100], 1, 64, 64, 64, False, 4)
    c.tables[0, 0] = c.nb + 5                 # held pooled blocks only: the window begins far behind it
    off, ctx, st = ints([0, 1]), ints([100]), status()
    q, out, scr, w = act(np.zeros((1, 64)), False), act(np.zeros((1, 64)), False), torch.empty(1 << 16, dtype=torch.uint8, device=DEV), c.window(1.0, 8, 0)
    check(lib.logismos_launch_window_attention_decode_bf16(P(q), 64, P(c.kp), P(c.vp), P(c.tables), P(ctx), P(off), P(out), 64, P(scr), 1, 1, 512, c.mb, c.nb, 1, 1, 64, C.byref(w), P(st), stream()), "d")
    torch.cuda.synchronize()
    assert st.item() == 1


# ---- differential attention ------------------------------------------------------------------------

def by_map(x, G):
    """[T, H, 2, d] -> [T, 2 H, d] in the order key head, map, query head of the key head."""
    T, H, _, d = x.shape
    return x.reshape(T, G, H // G, 2, d).transpose(0, 1, 3, 2, 4).reshape(T, 2 * H, d)


@pytest.mark.parametrize("H,G,D,d,v,size", [(6, 3, 64, 22, 30, 20), (20, 1, 64, 8, 8, 3), (4, 1, 128, 64, 128, 700), (2, 2, 256, 100, 200, 130)])
def test_differential_decode(H, G, D, d, v, size):
    rng = np.random.default_rng(H)
    lens = [1, 2, 16, 21, 150, 700]
    c, n, half, lam, eps = Cache(rng, lens, G, D, D, v, False), len(lens), D // 2, 0.45, 1e-3
    q = host(act(padded(rng.standard_normal((n, H, 2, d)), half), False))
    wide = np.zeros((n, H, 2, 2, half))
    wide[:, :, 0, 0], wide[:, :, 1, 1] = q[:, :, 0], q[:, :, 1]
    qd, scale = act(by_map(wide.reshape(n, H, 2, D), G).reshape(n, -1), False), 2.0 / np.sqrt(d)
    want = np.zeros((n, H, D))
    for s in range(n):
        maps = c.k[s].reshape(lens[s], G, 2, half)
        a = [R.attend(q[s:s + 1, :, m], maps[:, :, m], c.v[s], scale, R.chunk_mask(lens[s], size)[[lens[s] - 1]]) for m in range(2)]
        want[s, :, :v] = R.difference(a[0][..., :v], a[1][..., :v], lam, 0.2, eps)[0]
    for chunk in (64, 512):
        out = act(np.full((n, H * D + 8), 5.0), False)
        decode_call(c, qd, H, c.window(scale, size, 1), chunk, out, (v, lam, 0.8, eps))
        close(host(out)[:, :H * D].reshape(n, H, D), want, 1e-2)


@pytest.mark.parametrize("H,G,D,d,v,size,chunked", [(6, 3, 64, 22, 30, 20, 1), (20, 1, 64, 8, 8, 3, 1), (4, 1, 128, 64, 128, 700, 1), (2, 2, 128, 40, 100, 1, 1), (3, 1, 128, 64, 128, 130, 1),
                                                      (4, 2, 64, 32, 64, 200, 0), (2, 1, 128, 50, 128, 0, 0)])
def test_differential_prompts(H, G, D, d, v, size, chunked):
    """Both maps in one pass; one pair of keys in sight stands out in the first map alone and another in the second."""
    rng = np.random.default_rng(H + size)
    lens, new = [2, 130, 300, 700, 523, 411, 1], [2, 130, 2, 300, 129, 17, 1]
    c, n, half, lam, eps, T = Cache(rng, lens, G, D, D, v, False), len(lens), D // 2, 0.6, 1e-3, sum(new)
    assert lib.logismos_differential_has_prompts(D) and not lib.logismos_differential_has_prompts(256)
    q = padded(rng.standard_normal((T, H, 2, d)), half)
    cu = np.concatenate([[0], np.cumsum(new)]).astype(np.int32)
    for s in range(n):
        maps = c.k[s].reshape(lens[s], G, 2, half)
        for i in range(new[s]):
            p = lens[s] - new[s] + i
            first = (p - p % size if chunked else max(0, p - size + 1)) if size else 0
            for m, j in ((0, first), (1, max(first, p - 1))):
                q[cu[s] + i, 0, m, :d] += 1.5 * maps[j, 0, m, :d]
    q = host(act(q, False))
    wide = np.zeros((T, H, 2, 2, half))
    wide[:, :, 0, 0], wide[:, :, 1, 1] = q[:, :, 0], q[:, :, 1]
    qd, scale = act(by_map(wide.reshape(T, H, 2, D), G).reshape(T, -1), False), 1.0 / np.sqrt(d)
    want = np.zeros((T, H, D))
    for s in range(n):
        maps, rows = c.k[s].reshape(lens[s], G, 2, half), np.arange(lens[s] - new[s], lens[s])
        mask = (R.chunk_mask(lens[s], size) if chunked else R.window_mask(lens[s], size or lens[s]))[rows]
        a = [R.attend(q[cu[s]:cu[s + 1], :, m], maps[:, :, m], c.v[s], scale, mask) for m in range(2)]
        want[cu[s]:cu[s + 1], :, :v] = R.difference(a[0][..., :v], a[1][..., :v], lam, 0.2, eps)
    w, st = c.window(scale, size, chunked), status()
    keys = [lib.logismos_window_view_keys(C.byref(w), x, y) for x, y in zip(lens, new)]
    scr = torch.empty(lib.logismos_paged_prefix_attention_scratch_bytes(sum(keys), n, G, D), dtype=torch.uint8, device=DEV)
    scr.fill_(255)
    out, keep = act(np.full((T, H * D + 8), 5.0), False), [ints(cu), ints(lens)]
    check(lib.logismos_launch_differential_prefix_bf16(P(qd), 2 * H * D, P(keep[0]), P(keep[1]), P(c.kp), P(c.vp), P(c.tables), c.mb, c.nb, P(out), H * D + 8, P(scr), T, sum(keys), n, max(new),
                                                       max(keys), H, G, D, C.byref(w), v, lam, 0.8, eps, P(st), stream()), "prefix")
    torch.cuda.synchronize()
    assert st.item() == 0
    got = host(out)
    close(got[:, :H * D].reshape(T, H, D), want, 1e-2)
    assert (got[:, H * D:] == 5.0).all()


@FP32
@pytest.mark.parametrize("rows,H,G,v,vp_", [(1, 1, 1, 9, 64), (37, 6, 2, 30, 64), (300, 4, 4, 128, 128), (9, 20, 1, 200, 256)])
def test_difference_of_two_attentions(rows, H, G, v, vp_, fp32):
    rng = np.random.default_rng(rows)
    a = padded(rng.standard_normal((rows, H, 2, v)), vp_)
    ad, out = fl(np.concatenate([by_map(a, G).reshape(rows, -1), np.full((rows, 4), 9.0)], axis=1)), act(np.full((rows, H * vp_ + 8), 3.0), fp32)
    check(lib.logismos_launch_attention_difference(P(ad), ad.shape[1], P(out), H * vp_ + 8, int(fp32), rows, H, G, v, vp_, 0.6, 0.75, 1e-2, stream()), "difference")
    want = padded(R.difference(a[:, :, 0, :v], a[:, :, 1, :v], 0.6, 0.25, 1e-2), vp_).reshape(rows, -1)
    close(host(out)[:, :H * vp_], want, 1e-6 if fp32 else 3e-3)
    assert (host(out)[:, H * vp_:] == 3.0).all()


# ---- norms per head, rotation, cache, means of blocks ----------------------------------------------

@FP32
@pytest.mark.parametrize("H,G,maps,hd,dim,rot,pool", [(6, 2, 1, 64, 20, {"dims": 12, "base": 80.0}, 5), (4, 1, 1, 128, 128, {"dims": 64, "base": 5e4}, 16), (2, 2, 1, 256, 150, {"dims": 150, "base": 1e4}, 1),
                                                      (3, 3, 1, 32, 8, {"dims": 0, "base": 9.0}, 40), (6, 3, 2, 32, 22, {"dims": 6, "base": 300.0, "scaling": {"factor": 3.0}}, 0),
                                                      (4, 1, 2, 64, 64, {"dims": 64, "base": 1e4}, 3), (20, 1, 2, 128, 120, {"dims": 100, "base": 1e4}, 0)])
def test_norms_per_head_rotation_store_and_means(H, G, maps, hd, dim, rot, pool, fp32):
    """Decode rows that end blocks, and prompt rows of two sequences, one of which continues, in one step."""
    rng = np.random.default_rng(dim)
    U, eps, mb = maps * (H + 2 * G), 1e-3, 8
    spans = [(44, 45), (16, 17), (0, 1), (59, 60), (0, 70), (27, 97)]               # positions of each sequence in the step
    n_dec, rows = 4, sum(b - a for a, b in spans)
    perm = rng.permutation(len(spans) * mb)
    tables = perm.reshape(len(spans), mb).astype(np.int32)
    nb, width = perm.size, G * maps * hd
    pools = [act(rng.standard_normal((nb, 16, width)), fp32) for _ in range(2)]
    old = [host(p) for p in pools]
    mean_rows = -(-16 // pool) if pool else 1
    means = [act(np.full((nb, mean_rows, width), 7.0), fp32) for _ in range(2)]
    seq = np.concatenate([np.full(b - a, s) for s, (a, b) in enumerate(spans)])
    pos = np.concatenate([np.arange(a, b) for a, b in spans])
    slots = tables[seq, pos // 16].astype(np.int64) * 16 + pos % 16
    ld = U * hd + 24
    full = np.zeros((rows, ld))
    full[:, :U * hd] = padded(rng.standard_normal((rows, U, dim)), hd).reshape(rows, -1)
    src = act(full, fp32)
    full = host(src)
    gains = [padded(rng.standard_normal(dim), hd) for _ in range(2)]
    qx, st = act(np.full((rows, 4 * H * hd + 8), 3.0), fp32), status()
    keep = [fl(gains[0]), fl(gains[1]), angles(rot, 200) if rot["dims"] else None, dev(slots, torch.int64), ints(pos), ints(tables), ints(seq)]
    a = HeadNorm(qkv=A(src), ld=ld, rows=rows, heads=H, n_kv=G, maps=maps, hd=hd, dim=dim, gain_q=A(keep[0]), gain_k=A(keep[1]), eps=eps, table=A(keep[2]), rot_dims=rot["dims"], q_out=A(qx),
                 ld_q=4 * H * hd + 8, k_pool=A(pools[0]), v_pool=A(pools[1]), slots=A(keep[3]), positions=A(keep[4]), n_pool_slots=nb * 16, pool=pool, pool_rows=n_dec, k_mean=A(means[0]),
                 v_mean=A(means[1]), tables=A(keep[5]), seq_ids=A(keep[6]), max_blocks=mb, n_pool_blocks=nb)
    check(lib.logismos_launch_head_norm_store(C.byref(a), int(fp32), P(st), stream()), "store")
    if pool:
        check(lib.logismos_launch_pool_blocks(C.byref(a), int(fp32), P(st), stream()), "means")
    torch.cuda.synchronize()
    assert st.item() == 0
    x = full[:, :U * hd].reshape(rows, U, hd)
    nq, nk = maps * H, maps * G
    turn = lambda y, g: padded(R.rotate(R.rms(y[..., :dim], eps) * g[:dim], pos, rot, False) if rot["dims"] else R.rms(y[..., :dim], eps) * g[:dim], hd)
    q, k = turn(x[:, :nq], gains[0]), turn(x[:, nq:nq + nk], gains[1])
    tol = 1e-6 if fp32 else 3e-3
    if maps == 1:
        close(host(src)[:, :nq * hd].reshape(rows, nq, hd), q, tol)
    else:
        rep, wide = H // G, np.zeros((rows, G, 2, H // G, 2, hd))
        for m in range(2):
            wide[:, :, m, :, m] = q.reshape(rows, G, 2, rep, hd)[:, :, m]
        close(host(qx)[:, :4 * H * hd].reshape(wide.shape), wide, tol)
        assert (host(qx)[:, :4 * H * hd].reshape(wide.shape)[wide == 0] == 0).all() and np.array_equal(host(src), full)
    assert np.array_equal(host(src)[:, nq * hd:], full[:, nq * hd:])
    got = [host(p).reshape(-1, width) for p in pools]
    close(got[0][slots].reshape(rows, nk, hd), k, tol)
    assert np.array_equal(got[1][slots], x[:, nq + nk:].reshape(rows, -1))
    untouched = np.setdiff1d(np.arange(nb * 16), slots)
    assert all(np.array_equal(g[untouched], o.reshape(-1, width)[untouched]) for g, o in zip(got, old))
    if not pool:
        return
    want = [np.full((nb, mean_rows, width), 7.0) for _ in range(2)]
    for s, (first, end) in enumerate(spans):
        for b in range(first // pool, end // pool):
            e = (b + 1) * pool - 1
            if e < first:
                continue
            page = e // 16
            row = b - sum((j + 1) * pool - 1 < page * 16 for j in range(b))
            at = [tables[s, j // 16] * 16 + j % 16 for j in range(b * pool, e + 1)]
            for w, g in zip(want, got):
                w[tables[s, page], row] = g[at].mean(axis=0)
    for m, w in zip(means, want):
        close(host(m), w, 1e-6 if fp32 else 3e-3)
        assert np.array_equal(host(m) == 7.0, w == 7.0)
    keep[3].fill_(nb * 16)
    check(lib.logismos_launch_head_norm_store(C.byref(a), int(fp32), P(st), stream()), "store")
    torch.cuda.synchronize()
    assert st.item() == 1


# ---- residual ----------------------------------------------------------------------------------------

@FP32
@pytest.mark.parametrize("rows,n", [(1, 60), (5, 88), (70, 512), (700, 1000), (3, 4096), (2, 9000)])
def test_gated_residuals(rows, n, fp32):
    rng = np.random.default_rng(n)
    ld, eps, vocab = -(-n // 64) * 64, 1e-3, 50
    vec = lambda *s: padded(rng.standard_normal(s + (n,)), ld)
    x, ys, gains, step = vec(rows), [vec(rows), 0.1 * vec(rows)], [vec(), vec()], vec()
    gate_d, emb_d, ids = act(np.concatenate([2 * vec(rows), np.zeros((rows, 8))], axis=1), fp32), act(vec(vocab), False), rng.integers(0, vocab, rows)
    gate, emb = host(gate_d)[:, :ld], host(emb_d)
    pairs, top = 5, 3
    er, pr, wt = act(vec(rows * pairs + 1), fp32), rng.permutation(rows * pairs).reshape(rows, pairs), rng.uniform(0, 1, (rows, top))
    weights = np.concatenate([wt, np.ones((rows, pairs - top))], axis=1)
    counts = ints(np.ones(7))
    keep = [fl(g) for g in gains] + [fl(step), ints(ids), ints(pr), fl(wt)]
    mo = MixtureOut(A(er), A(keep[4]), A(keep[5]), 0, pairs, top, A(counts), 7)
    sig, true = R.sigmoid(gate), slice(0, n)
    mixed = (host(er)[pr] * weights[..., None]).sum(axis=1)
    two = 0.5 * sum(padded(R.rms(y[:, true], eps), ld) * g for y, g in zip(ys, gains))
    tol = 1e-6 if fp32 else 3e-3
    for name, y in (("none", 0.0 * x), ("one", ys[0]), ("two", two), ("mixture", mixed)):
        for enter in (False, True):
            xd, h, kept, st = fl(x), act(np.zeros((rows, ld)), fp32), fl(np.zeros((rows, ld))), status()
            yd = [fl(v) for v in ys]
            a = GatedResidual(x=A(xd), eps=eps, gain=1.3, n_src_rows=rows, rows=rows, n=n, ld=ld, is_f32=int(fp32), h=A(h), zero_branches=1, kept=A(kept))
            if name != "none":
                a.gate, a.ld_gate = A(gate_d), ld + 8
            if name in ("one", "two"):
                a.branch[0] = A(yd[0])
            if name == "two":
                a.branch[1], a.branch_gain[0], a.branch_gain[1] = A(yd[1]), A(keep[0]), A(keep[1])
            if name == "mixture":
                a.mixture = C.pointer(mo)
            if enter:
                a.embed, a.ids, a.vocab, a.step = A(emb_d), A(keep[3]), vocab, A(keep[2])
            check(lib.logismos_launch_gated_residual(C.byref(a), P(st), stream()), name)
            mid = x + y * sig if name != "none" else x
            want = mid + emb[ids] + step if enter else mid
            close(host(kept), mid, 2e-6)
            close(host(xd), want, 2e-6)
            close(host(h), padded(R.rms(want[:, true], eps), ld) * 1.3, tol)
            assert (host(h)[:, n:] == 0).all() and st.item() == 0
            assert (name in ("one", "two")) == (not yd[0].any()) and (name == "two") == (not yd[1].any())
    assert not counts.any()
    # rows picked; an index outside raises the status
    xd, idx, h, st = fl(x), rng.integers(0, rows, 5), act(np.zeros((5, ld)), fp32), status()
    a = GatedResidual(x=A(xd), eps=eps, gain=0.5, n_src_rows=rows, rows=5, n=n, ld=ld, is_f32=int(fp32), h=A(h))
    picked = ints(idx)
    a.row_idx = A(picked)
    check(lib.logismos_launch_gated_residual(C.byref(a), P(st), stream()), "pick")
    close(host(h), padded(R.rms(x[idx][:, true], eps), ld) * 0.5, tol)
    assert st.item() == 0
    picked.fill_(rows)
    check(lib.logismos_launch_gated_residual(C.byref(a), P(st), stream()), "pick")
    torch.cuda.synchronize()
    assert st.item() == 1


# ---- linear attention --------------------------------------------------------------------------------

def run_linear(form, heads, dk, dv, lens, seed, fp32=False, decays=None):
    """Two calls over ragged sequences, the second continuing the first in other slots' company."""
    rng = np.random.default_rng(seed)
    pad = lambda d: max(32, 1 << (d - 1).bit_length())
    dp, wp, n = pad(dk), pad(dv), len(lens)
    decay = np.linspace(0.4, 0.9995, heads) if decays is None else np.asarray(decays)
    state, sl, S = fl(np.full((n + 2, heads, dp, wp), np.nan)), rng.permutation(n + 2)[:n], [np.zeros((heads, dk, dv)) for _ in lens]
    parts = fl(np.stack([np.maximum(np.log2(np.maximum(decay, 1e-300)), -1e4), decay, decay - decay.astype(np.float32)], axis=1))
    outs, wants = [], []
    for call in range(2):
        ll = lens if call == 0 else lens[::-1]
        T, cu = sum(ll), np.concatenate([[0], np.cumsum(ll)]).astype(np.int32)
        v, k, q = rng.standard_normal((T, heads, dv)), rng.standard_normal((T, heads, dk)) / np.sqrt(dk), rng.standard_normal((T, heads, dk))
        rows = act(np.concatenate([np.zeros((T, 8)), padded(v, wp).reshape(T, -1), padded(k, dp).reshape(T, -1), padded(q, dp).reshape(T, -1), np.zeros((T, 24))], axis=1), fp32)
        r = host(rows)[:, 8:8 + heads * (wp + 2 * dp)]
        v, k, q = r[:, :heads * wp].reshape(T, heads, wp)[..., :dv], r[:, heads * wp:heads * (wp + dp)].reshape(T, heads, dp)[..., :dk], r[:, heads * (wp + dp):].reshape(T, heads, dp)[..., :dk]
        out, keep = act(np.full((T, heads * wp + 8), 4.0), fp32), [ints(sl), dev(np.full(n, call == 0, np.uint8), torch.uint8), ints(cu)]
        a = Ssd(state=A(state), state_slots=A(keep[0]), fresh=A(keep[1]), cu=A(keep[2]), y=A(out), ld_y=heads * wp + 8, heads=heads, groups=heads, np=dp, vp=wp,
                xbc=A(rows) + 8 * (4 if fp32 else 2), ld_xbc=rows.shape[1], decay=A(parts))
        if form == "chunked":
            check(lib.logismos_launch_ssd_chunked_bf16(C.byref(a), n, stream()), "chunked")
        elif form == "segments":
            entries = T // 256 + n + 1
            scr = torch.full((lib.logismos_ssd_scratch_bytes(entries, heads, dp, wp) // 4,), float("nan"), device=DEV)
            check(lib.logismos_launch_ssd_segmented_bf16(C.byref(a), n, max(ll), P(scr), entries, stream()), "segments")
        else:
            check(lib.logismos_launch_ssd_step(C.byref(a), n, int(fp32), stream()), "step")
        want = np.zeros((T, heads, dv))
        for s in range(n):
            i = slice(cu[s], cu[s + 1])
            for h in range(heads):
                want[i, h], S[s][h] = R.decay_recurrence(q[i, h], k[i, h], v[i, h], decay[h], S[s][h])
        o = host(out)[:, :heads * wp].reshape(T, heads, wp)
        assert (o[..., dv:] == 0).all()
        outs.append(o[..., :dv])
        wants.append(want)
    st = host(state)[sl]
    assert (st[:, :, dk:] == 0).all() and (st[..., dv:] == 0).all()
    return np.concatenate(outs), np.concatenate(wants), st[:, :, :dk, :dv], np.stack(S)


@pytest.mark.parametrize("heads,dk,dv", [(3, 24, 40), (2, 64, 128), (5, 10, 8), (2, 128, 64)])
@pytest.mark.parametrize("lens", [[1, 2, 63, 64, 65], [200, 15], [129]])
def test_linear_attention_with_a_fixed_decay(heads, dk, dv, lens):
    for form, fp32, tol in (("chunked", False, 4e-3), ("step", False, 4e-3), ("step", True, 2e-6)):
        o, want, st, S = run_linear(form, heads, dk, dv, lens, 7, fp32)
        close(o, want, tol)
        close(st, S, 1e-4 if form == "chunked" else 1e-5)


@pytest.mark.parametrize("heads,dk,dv", [(3, 24, 40), (1, 64, 128), (2, 128, 16)])
@pytest.mark.parametrize("lens", [[1500], [256, 257, 3, 255, 700], [511, 512, 513]])
def test_segments_of_long_prompts(heads, dk, dv, lens):
    for decays in (None, [0.9999] * heads, [0.0] * heads):
        o, want, st, S = run_linear("segments", heads, dk, dv, lens, 3, decays=decays)
        close(o, want, 4e-3)
        close(st, S, 1e-4)
    assert lib.logismos_ssd_segments(1500, 1, 1500, 8) == 1500 // 256 + 2
    assert lib.logismos_ssd_segments(1500, 3, 512, 8) == 0 and lib.logismos_ssd_segments(4096, 4, 1024, 32) == 0 and lib.logismos_ssd_segments(16384, 1, 16384, 32) > 0


def test_linear_attention_at_the_ends_of_the_decay_and_in_large_heads():
    for form in ("chunked", "step"):
        o, want, st, S = run_linear(form, 3, 40, 32, [130, 3, 64], 5, decays=[1.0, 0.0, 1e-9])
        close(o, want, 4e-3)
        close(st, S, 1e-4)
    o, want, st, S = run_linear("step", 2, 136, 200, [1, 30], 6)
    close(o, want, 4e-3)
    assert not lib.logismos_ssd_has_chunked(256, 32)


@FP32
@pytest.mark.parametrize("rows,heads,v,vp_", [(1, 3, 40, 64), (70, 4, 64, 64), (9, 5, 8, 32), (300, 16, 128, 128), (3, 40, 128, 128), (2, 80, 128, 128)])
def test_norm_over_all_heads_and_gate(rows, heads, v, vp_, fp32):
    rng = np.random.default_rng(rows)
    y, z = (act(padded(rng.standard_normal((rows, heads, v)), vp_).reshape(rows, -1), fp32) for _ in range(2))
    gain, out = padded(rng.standard_normal((heads, v)), vp_), act(np.zeros((rows, heads * vp_ + 8)), fp32)
    gd = fl(gain.reshape(-1))
    check(lib.logismos_launch_norm_gate(P(y), heads * vp_, P(z), heads * vp_, P(gd), P(out), heads * vp_ + 8, int(fp32), rows, heads, v, vp_, 1e-3, stream()), "gate")
    true = lambda t: host(t).reshape(rows, heads, vp_)[..., :v].reshape(rows, -1)
    want = R.rms(true(y), 1e-3) * gain[:, :v].reshape(-1) * R.sigmoid(true(z))
    close(true(out[:, :heads * vp_]), want, 2e-6 if fp32 else 4e-3)


# ---- projections with silu, clamped experts, router ---------------------------------------------------

@pytest.mark.parametrize("m", [1, 20, 60, 130, 600])
def test_projections_with_silu_columns_and_a_bias(m):
    rng = np.random.default_rng(m)
    K, n_main, n_tail, silu = 192, 640, 16, (96, 352)
    n = n_main + n_tail
    a, w, b = act(rng.standard_normal((m, K)), False), act(rng.standard_normal((n, K)) / np.sqrt(K), False), rng.standard_normal(n_main)
    z = host(a) @ host(w).T
    z[:, :n_main] += b
    want = z.copy()
    want[:, silu[0]:silu[1]] = R.silu(z[:, silu[0]:silu[1]])
    bd = fl(b)

    def run(form):
        out, tail, st = act(np.zeros((m, n_main)), form == "f32"), fl(np.zeros((m, n_tail))), status()
        g = Groups(1, (i32 * 8)(n), n_main, A(tail), n_tail, 0.0, 0, A(bd), *silu)
        if form == "f32":
            af = fl(host(a))
            check(lib.logismos_launch_linear_groups_f32(P(af), P(w), P(out), m, n, K, K, n_main, C.byref(g), stream()), form)
        elif form == "small":
            check(lib.logismos_launch_linear_groups_small_bf16(P(a), P(w), P(out), m, n, K, K, n_main, C.byref(g), stream()), form)
        elif form == "tiles":
            check(lib.logismos_launch_linear_groups_tc_bf16(P(a), P(w), P(out), m, n, K, K, n_main, C.byref(g), P(st), stream()), form)
        else:
            acc = fl(np.zeros((m, n)))
            check(lib.logismos_launch_linear_t_act_bf16(P(a), P(w), P(None), P(acc), m, n, K, K, n, 0x101, 0, 0, 0, P(st), stream()), form)
            check(lib.logismos_launch_linear_groups_finish(P(acc), P(out), m, n, n, n_main, C.byref(g), stream()), form)
            assert not acc.any()
        close(host(out), want[:, :n_main], 2e-6 if form == "f32" else 3e-3)
        close(host(tail), want[:, n_main:], 2e-6 if form == "f32" else 1e-5)
        assert st.item() == 0
    for form in ("f32", "small", "tiles", "sums"):
        run(form)
    bad = Groups(1, (i32 * 8)(n), n_main, A(bd), n_tail, 0.0, 0, A(bd), 16, 64)
    assert lib.logismos_launch_linear_groups_f32(P(bd), P(w), P(bd), 1, n, K, K, n_main, C.byref(bad), stream())


@pytest.mark.parametrize("form", ["few", "many", "f32"])
@pytest.mark.parametrize("E,top,count,keep,tokens", [(6, 2, 3, 2, 5), (16, 3, 4, 2, 40), (12, 1, 4, 1, 33), (3, 3, 1, 1, 7), (4, 2, 4, 2, 20), (40, 4, 8, 3, 61), (130, 6, 10, 4, 64), (512, 8, 16, 4, 30)])
def test_mixture_by_groups_with_clamped_units(E, top, count, keep, tokens, form):
    rng = np.random.default_rng(E + tokens)
    H, F, limit = 64, 64, 0.7
    if form == "many":
        tokens *= 9
    fp32 = form == "f32"
    ld = -(-E // 16) * 16
    z = 2 * rng.standard_normal((tokens, ld))
    zd, hd = fl(z), act(rng.standard_normal((tokens, H)), fp32)
    gate, upw, down = (host(act(rng.standard_normal((E, F, H)) / 8, False)) for _ in range(3))
    inter = np.zeros((E, 2 * F, H))
    for b in range(F // 32):
        inter[:, 64 * b:64 * b + 32], inter[:, 64 * b + 32:64 * b + 64] = gate[:, 32 * b:32 * b + 32], upw[:, 32 * b:32 * b + 32]
    wu, wd = act(inter.reshape(-1, H), False), act(down.transpose(0, 2, 1).reshape(-1, F), False)
    it = lambda *s: torch.zeros(s, dtype=torch.int32, device=DEV)
    wts, prow, ident, off, tok, counts, pe = fl(np.zeros((tokens, top))), it(tokens, top), fl(np.zeros(tokens)), it(E + 1), it(tokens * top), it(E), it(tokens, top)
    mt = lib.logismos_moe_max_tiles(tokens, top, E, 0)
    tiles, nt, gat, st = it(mt, 4), it(1), act(np.zeros((tokens * top, H)), False), status()
    r = MoeRoute(A(zd), ld, 0, 0, E, 0, top, 0, A(wts), A(prow), A(ident))
    r.scoring, r.groups, r.keep_groups = 1, count, keep
    mid, rows = act(np.zeros((tokens * top, F)), fp32), act(np.zeros((tokens * top, H)), fp32)
    if form == "many":
        r.counts, r.pair_expert, r.tiles, r.n_tiles = A(counts), A(pe), A(tiles), A(nt)
    else:
        r.offsets, r.row_token = A(off), A(tok)
    check(lib.logismos_launch_moe_route(C.byref(r), tokens, stream()), "route")
    if form == "few":
        check(lib.logismos_launch_linear_experts_small_bf16(P(hd), P(wu), P(mid), P(off), P(tok), E, tokens, 16, 2 * F, H, H, F, 4, 1.702, limit, 1.0, stream()), "up")
        check(lib.logismos_launch_linear_experts_small_bf16(P(mid), P(wd), P(rows), P(off), P(None), E, tokens, 16, H, F, F, H, 0, 0, 0, 0, stream()), "down")
    elif form == "f32":
        check(lib.logismos_launch_linear_experts_f32(P(hd), P(wu), P(mid), P(off), P(tok), E, tokens, 2 * F, H, H, F, 4, 1.702, limit, 1.0, stream()), "up")
        check(lib.logismos_launch_linear_experts_f32(P(mid), P(wd), P(rows), P(off), P(None), E, tokens, H, F, F, H, 3, 0, 0, 0, stream()), "down")
    else:
        check(lib.logismos_launch_moe_place(C.byref(r), P(hd), P(gat), H, tokens, stream()), "place")
        check(lib.logismos_launch_linear_experts_tc_bf16(P(gat), tokens * top, P(None), 0, P(wu), P(mid), P(tiles), P(nt), mt, E, 2 * F, H, H, F, 4, 1.702, limit, 1.0, P(st), stream()), "up")
        check(lib.logismos_launch_linear_experts_tc_bf16(P(mid), tokens * top, P(None), 0, P(wd), P(rows), P(tiles), P(nt), mt, E, H, F, F, H, 0, 0, 0, 0, P(st), stream()), "down")
    torch.cuda.synchronize()
    assert st.item() == 0
    chosen, weight = R.route(host(zd)[:, :E], top, count, keep)
    close(host(wts), weight, 1e-5)
    p = prow.cpu().numpy()
    assert sorted(p.reshape(-1).tolist()) == list(range(tokens * top))
    h, o = host(hd), host(rows)
    want = np.stack([[R.clamped_unit(h[t], {"gate": gate[e], "up": upw[e], "down": down[e].T}, limit) for e in chosen[t]] for t in range(tokens)])
    close(o[p], want, 2e-6 if fp32 else 8e-3)


def test_launchers_reject_what_they_cannot_run():
    x, st = fl(np.zeros((64, 256))), status()
    bad = lambda w: lib.logismos_launch_window_attention_f32(P(x), 64, P(x), P(x), P(st), P(st), P(st), P(x), 64, 1, 1, 1, 1, 1, 64, C.byref(w), P(st), stream())
    for w in (Window(scale=1.0, size=0, chunked=1), Window(scale=1.0, size=4, chunked=1, pool=2, k_mean=A(x), v_mean=A(x)), Window(scale=1.0, size=4, pool=2),
              Window(scale=1.0, size=4, pool=2, keep_first=1, k_mean=A(x), v_mean=A(x)), Window(scale=1.0, size=4, pool=-1)):
        assert bad(w)
    a = HeadNorm(qkv=A(x), ld=256, rows=1, heads=2, n_kv=1, maps=1, hd=48, dim=8, gain_q=A(x), gain_k=A(x), k_pool=A(x), v_pool=A(x), slots=A(x), positions=A(x), n_pool_slots=1)
    assert lib.logismos_launch_head_norm_store(C.byref(a), 1, P(st), stream())
    a.hd, a.maps, a.ld = 32, 2, 256
    assert lib.logismos_launch_head_norm_store(C.byref(a), 1, P(st), stream())          # nowhere to put the queries
    a.maps, a.pool = 1, 4
    assert lib.logismos_launch_head_norm_store(C.byref(a), 1, P(st), stream())          # nor the means
    assert lib.logismos_launch_attention_difference(P(x), 256, P(x), 256, 1, 1, 2, 1, 65, 64, 0.1, 1.0, 1e-6, stream())
    g = GatedResidual(x=A(x), rows=1, n_src_rows=1, n=64, ld=64, is_f32=1, h=A(x), gain=1.0)
    g.branch[0] = A(x)
    assert lib.logismos_launch_gated_residual(C.byref(g), P(st), stream())              # a sublayer without its gate
    r = MoeRoute(A(x), 16, 0, 0, 8, 0, 3, 0, A(x), A(x), A(x), A(x), A(x))
    r.scoring, r.groups, r.keep_groups = 1, 4, 1
    assert lib.logismos_launch_moe_route(C.byref(r), 1, stream())                        # three of a group of two
    r.groups, r.keep_groups, r.top = 3, 1, 2
    assert lib.logismos_launch_moe_route(C.byref(r), 1, stream())
    s = Ssd(state=A(x), state_slots=A(x), fresh=A(x), cu=A(x), y=A(x), ld_y=64, heads=1, groups=1, np=48, vp=64, xbc=A(x), ld_xbc=256, decay=A(x))
    assert lib.logismos_launch_ssd_step(C.byref(s), 1, 1, stream())
