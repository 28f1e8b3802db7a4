"""The kernels of the Vugedra decoder, each against the plain function of vugedra_reference.py."""
import ctypes as C

import numpy as np
import pytest
import torch

import vugedra_reference as R
from logismos_b200._lib import check, lib
from logismos_b200.structs import Groups, LatentRotary, MixtureOut, MoeRoute, TanhNorm, TimeMix, Window

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


def act(a, fp32):
    return fl(a) if fp32 else dev(np.asarray(a, np.float32), torch.bfloat16)


def close(got, want, tol):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    err = np.sqrt(np.mean((got - want) ** 2)) / np.sqrt(np.mean(want ** 2))
    assert err <= tol and np.abs(got - want).max() <= 12 * tol * np.abs(want).max(), (err, np.abs(got - want).max(), np.abs(want).max())


def angles(rot, positions):
    f, amp = R.rotary_frequencies(rot)
    a = np.arange(positions)[:, None] * f
    return fl(np.stack([amp * np.cos(a), amp * np.sin(a)], axis=-1).reshape(positions, -1))


def status():
    return torch.zeros(1, dtype=torch.int32, device=DEV)


# ---- tanh norms ------------------------------------------------------------------------------------

def tanh_vectors(rng, n, ld):
    w, b = np.zeros(ld), np.zeros(ld)
    w[:n], b[:n] = rng.standard_normal(n), rng.standard_normal(n)
    return float(np.float32(rng.uniform(0.3, 2.0))), w, b


@pytest.mark.parametrize("rows,n", [(1, 60), (3, 88), (70, 512), (1300, 1000)])
@pytest.mark.parametrize("fp32", [False, True])
def test_tanh_norms_and_residual(rows, n, fp32):
    rng = np.random.default_rng(n)
    ld = -(-n // 64) * 64
    x, y = np.zeros((rows, ld)), np.zeros((rows, ld))
    x[:, :n], y[:, :n] = 3 * rng.standard_normal((rows, n)), rng.standard_normal((rows, n))
    post, nxt = tanh_vectors(rng, n, ld), tanh_vectors(rng, n, ld)
    keep = [[fl(v) for v in p[1:]] for p in (post, nxt)]
    tp, tn = (TanhNorm(p[0], A(k[0]), A(k[1])) for p, k in zip((post, nxt), keep))
    xd, yd, hd, st = fl(x), fl(y), act(np.zeros((rows, ld)), fp32), status()
    check(lib.logismos_launch_tanh_norm(P(yd), 1, None, P(None), rows, P(xd), C.byref(tp), P(hd), C.byref(tn), int(fp32), rows, ld, P(st), stream()), "norm")
    want = x + R.tanh_norm(y, *post)
    close(host(xd), want, 1e-6)
    close(host(hd), R.tanh_norm(want, *nxt), 1e-6 if fp32 else 3e-3)
    assert not yd.any() and (host(xd)[:, n:] == 0).all() and (host(hd)[:, n:] == 0).all()
    # rows picked, no residual; an index outside raises the status
    idx = rng.integers(0, rows, 5)
    out = act(np.zeros((5, ld)), fp32)
    check(lib.logismos_launch_tanh_norm(P(None), 0, None, P(ints(idx)), rows, P(xd), None, P(out), C.byref(tn), int(fp32), 5, ld, P(st), stream()), "pick")
    close(host(out), R.tanh_norm(want[idx], *nxt), 1e-6 if fp32 else 3e-3)
    assert st.item() == 0
    check(lib.logismos_launch_tanh_norm(P(None), 0, None, P(ints([0, rows])), rows, P(xd), None, P(out), C.byref(tn), int(fp32), 2, ld, P(st), stream()), "pick")
    torch.cuda.synchronize()
    assert st.item() == 1


# ---- rotations -------------------------------------------------------------------------------------

@pytest.mark.parametrize("heads,kv,dim,hd,rot", [(6, 2, 20, 64, {"dims": 12, "base": 80.0, "scaling": {"factor": 2.5, "original": 30, "fast": 4.0, "slow": 0.7}}),
                                                 (4, 1, 128, 128, {"dims": 64, "base": 5e4}), (3, 3, 150, 256, {"dims": 150, "base": 1e4}), (2, 1, 8, 64, {"dims": 2, "base": 9.0})])
@pytest.mark.parametrize("fp32", [False, True])
def test_query_key_norm_rotation_and_store(heads, kv, dim, hd, rot, fp32):
    rng = np.random.default_rng(dim)
    rows, blocks, eps = 21, 4, 1e-3
    pos = rng.integers(0, 900, rows)
    slots = rng.permutation(blocks * 16)[:rows]
    ld = (heads + 2 * kv) * hd + 24
    full = np.zeros((rows, ld))
    cols = [h * hd + d for h in range(heads + 2 * kv) for d in range(dim)]
    full[:, cols] = rng.standard_normal((rows, len(cols)))
    src = act(full, fp32)
    full = host(src)
    gq, gk = np.zeros(heads * hd), np.zeros(kv * hd)
    gq.reshape(heads, hd)[:, :dim], gk.reshape(kv, hd)[:, :dim] = rng.standard_normal((heads, dim)), rng.standard_normal((kv, dim))
    pools = [act(np.zeros((blocks, 16, kv * hd)), fp32) for _ in range(2)]
    st, keep = status(), [fl(gq), fl(gk), angles(rot, 900), dev(slots.astype(np.int64), torch.int64), ints(pos)]
    go = lambda sl: check(lib.logismos_launch_qk_norm_rotary_store(P(src), ld, P(pools[0]), P(pools[1]), P(sl), P(keep[4]), rows, heads, kv, hd, dim, P(keep[0]),
                                                                   P(keep[1]), eps, P(keep[2]), rot["dims"], blocks * 16, int(fp32), P(st), stream()), "store")
    go(keep[3])
    part = lambda at, n: full[:, at * hd:(at + n) * hd].reshape(rows, n, hd)[..., :dim].reshape(rows, -1)
    norm = lambda x, g, n: R.rms_norm(x, g.reshape(n, hd)[:, :dim].reshape(-1), eps).reshape(rows, n, dim)
    q, k = R.rotate(norm(part(0, heads), gq, heads), pos, rot), R.rotate(norm(part(heads, kv), gk, kv), pos, rot)
    got = host(src)
    tol = 1e-6 if fp32 else 3e-3
    close(got[:, :heads * hd].reshape(rows, heads, hd)[..., :dim], q, tol)
    assert (got[:, :heads * hd].reshape(rows, heads, hd)[..., dim:] == 0).all()
    stored = [host(p).reshape(-1, kv, hd)[slots] for p in pools]
    close(stored[0][..., :dim], k, tol)
    assert np.array_equal(stored[1], full[:, (heads + kv) * hd:(heads + 2 * kv) * hd].reshape(rows, kv, hd))
    assert st.item() == 0 and np.array_equal(got[:, heads * hd:], full[:, heads * hd:])
    go(dev(np.full(rows, blocks * 16, np.int64), torch.int64))
    torch.cuda.synchronize()
    assert st.item() == 1


@pytest.mark.parametrize("heads,hd,at,dims", [(3, 64, 24, 6), (2, 128, 64, 64), (1, 256, 0, 250)])
@pytest.mark.parametrize("fp32", [False, True])
def test_rotation_of_a_part_of_every_head(heads, hd, at, dims, fp32):
    rng = np.random.default_rng(hd)
    rot, rows = {"dims": dims, "base": 1e3}, 13
    pos = rng.integers(0, 500, rows)
    q = act(rng.standard_normal((rows, heads * hd)), fp32)
    x, tab, ps = host(q).reshape(rows, heads, hd), angles(rot, 500), ints(pos)
    check(lib.logismos_launch_rotary_heads(P(q), heads * hd, P(ps), rows, heads, hd, at, P(tab), dims, int(fp32), stream()), "rotate")
    want = x.copy()
    want[..., at:at + dims] = R.rotate(x[..., at:at + dims], pos, rot)
    close(host(q).reshape(rows, heads, hd), want, 1e-6 if fp32 else 3e-3)


@pytest.mark.parametrize("q_n,c_n,dims,heads", [(27, 21, 6, 3), (80, 64, 16, 20), (130, 300, 100, 2), (16, 8, 2, 1)])
@pytest.mark.parametrize("fp32", [False, True])
def test_latent_rows_with_a_rotated_part(q_n, c_n, dims, heads, fp32):
    rng = np.random.default_rng(q_n)
    up = lambda v, to: -(-v // to) * to
    rows, blocks, eps, rot = 19, 3, 1e-3, {"dims": dims, "base": 300.0, "scaling": {"factor": 3.0, "original": 40, "fast": 8.0, "slow": 1.0}}
    qw, at = up(q_n, 64), up(c_n, 8)
    cw, lg = up(at + dims, 64), up(heads, 16)
    ld = qw + cw + lg
    raw = np.zeros((rows, ld))
    raw[:, :q_n], raw[:, qw:qw + c_n], raw[:, qw + at:qw + at + dims] = (rng.standard_normal((rows, n)) for n in (q_n, c_n, dims))
    raw[:, qw + cw:qw + cw + heads] = rng.standard_normal((rows, heads))
    gq, gc = np.zeros(qw), np.zeros(cw)
    gq[:q_n], gc[:c_n] = rng.standard_normal(q_n), rng.standard_normal(c_n)
    pos, slots = rng.integers(0, 700, rows), rng.permutation(blocks * 16)[:rows]
    keep = [angles(rot, 700), ints(pos), fl(gq), fl(gc), dev(slots.astype(np.int64), torch.int64)]
    rd, cq, pool, gate, st = fl(raw), act(np.zeros((rows, qw)), fp32), act(np.zeros((blocks, 16, cw)), fp32), fl(np.zeros((rows, lg))), status()
    lr = LatentRotary(A(keep[0]), A(keep[1]), at, dims, A(gate), heads, lg)
    check(lib.logismos_launch_latent_norm_store(P(rd), ld, P(keep[2]), P(keep[3]), P(cq), P(pool), P(keep[4]), rows, qw, q_n, cw, c_n, eps, blocks * 16, int(fp32), 1,
                                                C.byref(lr), P(st), stream()), "store")
    tol = 1e-6 if fp32 else 3e-3
    close(host(cq)[:, :q_n], R.rms_norm(raw[:, :q_n], gq[:q_n], eps), tol)
    got = host(pool).reshape(-1, cw)[slots]
    close(got[:, :c_n], R.rms_norm(raw[:, qw:qw + c_n], gc[:c_n], eps), tol)
    close(got[:, at:at + dims], R.rotate(raw[:, None, qw + at:qw + at + dims], pos, rot)[:, 0], tol)
    assert (got[:, c_n:at] == 0).all() and (got[:, at + dims:] == 0).all() and not rd.any() and st.item() == 0
    assert np.array_equal(host(gate)[:, :heads], raw[:, qw + cw:qw + cw + heads].astype(np.float32))


# ---- windowed attention ----------------------------------------------------------------------------

class Cache:
    """Sequences with random keys and values in shuffled pages, and the plain attention of any of their rows."""

    def __init__(self, rng, lens, H, G, D, dim, fp32, spare=3):
        self.H, self.G, self.D, self.lens, self.fp32 = H, G, D, lens, fp32
        self.mb = max(-(-n // 16) for n in lens) + 1
        self.nb = sum(-(-n // 16) for n in lens) + spare
        perm, at = rng.permutation(self.nb), 0
        tables = -np.ones((len(lens), self.mb), np.int32)
        pools = [np.full((self.nb, 16, G * D), np.nan) for _ in range(2)]   # what no sequence owns must not be touched
        self.k, self.v = [], []
        for s, n in enumerate(lens):
            b = -(-n // 16)
            tables[s, :b] = perm[at:at + b]
            at += b
            for pool, store in zip(pools, (self.k, self.v)):
                x = np.zeros((n, G, D))
                x[..., :dim] = rng.standard_normal((n, G, dim))
                x = host(act(x, fp32))
                store.append(x)
                for t in range(n):
                    pool[tables[s, t // 16], t % 16] = x[t].reshape(-1)
        self.tables = ints(tables)
        self.kp, self.vp = (act(p, fp32) for p in pools)

    def want(self, s, rows, q, scale, size, keep, sink, gate):
        """rows: positions; q [n, H, D]; gate [n, H]."""
        out = np.zeros((len(rows), self.H, self.D))
        for i, p in enumerate(rows):
            j = np.arange(p + 1)
            seen = (p - j < size) | (j < keep) if size else np.ones(p + 1, bool)
            for a in range(self.H):
                g = a // (self.H // self.G)
                z = np.where(seen, self.k[s][:p + 1, g] @ q[i, a] * scale, -np.inf)
                w = R.softmax_plus_one(z) if sink else R.softmax(z)
                out[i, a] = w @ self.v[s][:p + 1, g] * R.sigmoid(gate[i, a])
        return out


WINDOWS = [(1, 0, 1), (16, 5, 1), (17, 16, 0), (40, 130, 1), (128, 3, 1), (130, 129, 1), (200, 260, 1), (0, 0, 0), (1000, 4, 1)]


@pytest.mark.parametrize("size,keep,sink", WINDOWS)
@pytest.mark.parametrize("H,G,D,dim", [(6, 2, 64, 20), (20, 1, 64, 64), (4, 4, 128, 100), (2, 1, 256, 200)])
def test_window_attention_of_decoded_tokens(H, G, D, dim, size, keep, sink):
    rng = np.random.default_rng(size + keep)
    lens = [1, 2, 15, 16, 17, 33, 130, 145, 146, 300, 700]
    c = Cache(rng, lens, H, G, D, dim, False)
    n, ld, scale = len(lens), H * D + 16, 1.3 / np.sqrt(dim)
    q = np.zeros((n, ld))
    q[:, :H * D].reshape(n, H, D)[..., :dim] = rng.standard_normal((n, H, dim))
    qd, gate = act(q, False), rng.standard_normal((n, H + 2))
    q = host(qd)[:, :H * D].reshape(n, H, D)
    gd, st = fl(gate), status()
    w = Window(scale, size, keep, sink, A(gd), H + 2)
    ctx = np.array(lens, np.int32)
    for chunk in (64, 512):
        vctx = np.array([lib.logismos_window_context(v, size, keep) for v in lens], np.int32)
        off = np.empty(n + 1, np.int32)
        total = lib.logismos_build_decode_chunks(vctx.ctypes.data_as(vp), n, chunk, off.ctypes.data_as(vp))
        scr = torch.empty(max(1, lib.logismos_paged_decode_scratch_bytes(total, H, D)), dtype=torch.uint8, device=DEV)
        out, keepd = act(np.zeros((n, H * D + 8)), False), [ints(ctx), ints(off)]
        check(lib.logismos_launch_window_attention_decode_bf16(P(qd), ld, P(c.kp), P(c.vp), P(c.tables), P(keepd[0]), P(keepd[1]), P(out), H * D + 8, P(scr), n, total, chunk,
                                                               c.mb, c.nb, H, G, D, C.byref(w), P(st), stream()), "decode")
        got = host(out)[:, :H * D].reshape(n, H, D)
        want = np.concatenate([c.want(s, [lens[s] - 1], q[s:s + 1], scale, size, keep, sink, gate[s:s + 1]) for s in range(n)])
        close(got, want, 6e-3)
        assert st.item() == 0


@pytest.mark.parametrize("size,keep,sink", WINDOWS)
@pytest.mark.parametrize("H,G,D,dim", [(6, 2, 64, 20), (4, 4, 128, 100), (2, 1, 256, 200)])
def test_window_attention_of_prompts(H, G, D, dim, size, keep, sink):
    rng = np.random.default_rng(size + keep + 1)
    lens, new = [2, 130, 300, 700, 523, 411], [2, 130, 2, 300, 129, 17]
    c = Cache(rng, lens, H, G, D, dim, False)
    T, ld, scale, n = sum(new), H * D, 1.3 / np.sqrt(dim), len(lens)
    q = np.zeros((T, H, D))
    q[..., :dim] = rng.standard_normal((T, H, dim))
    qd, gate = act(q.reshape(T, -1), False), rng.standard_normal((T, H))
    q, gd, st = host(qd).reshape(T, H, D), fl(gate), status()
    cu = np.concatenate([[0], np.cumsum(new)]).astype(np.int32)
    keys = [lib.logismos_window_keys(a, b, size, keep) for a, b in zip(lens, new)]
    scr = torch.empty(lib.logismos_paged_prefix_attention_scratch_bytes(sum(keys), n, G, D), dtype=torch.uint8, device=DEV)
    scr.fill_(255)
    out, keepd, w = act(np.zeros((T, ld + 8)), False), [ints(cu), ints(lens)], Window(scale, size, keep, sink, A(gd), H)
    check(lib.logismos_launch_window_attention_prefix_bf16(P(qd), ld, P(keepd[0]), P(keepd[1]), P(c.kp), P(c.vp), P(c.tables), c.mb, c.nb, P(out), ld + 8, P(scr), T, sum(keys), n,
                                                           max(new), max(keys), H, G, D, C.byref(w), P(st), stream()), "prefix")
    got = host(out)[:, :ld].reshape(T, H, D)
    rows = lambda s: np.arange(lens[s] - new[s], lens[s])
    want = np.concatenate([c.want(s, rows(s), q[cu[s]:cu[s + 1]], scale, size, keep, sink, gate[cu[s]:cu[s + 1]]) for s in range(n)])
    close(got, want, 6e-3)
    assert st.item() == 0


@pytest.mark.parametrize("size,keep,sink", WINDOWS)
def test_window_attention_f32(size, keep, sink):
    rng = np.random.default_rng(size + keep + 2)
    H, G, D, dim, lens = 6, 3, 64, 40, [1, 65, 300]
    c = Cache(rng, lens, H, G, D, dim, True)
    rows = [(s, p) for s, n in enumerate(lens) for p in sorted({0, n // 2, n - 1})]
    T = len(rows)
    q = np.zeros((T, H, D))
    q[..., :dim] = rng.standard_normal((T, H, dim))
    qd, gate = fl(q.reshape(T, -1)), rng.standard_normal((T, H))
    gd, st, out = fl(gate), status(), fl(np.zeros((T, H * D)))
    w, keepd = Window(0.2, size, keep, sink, A(gd), H), [ints([r[0] for r in rows]), ints([r[1] for r in rows])]
    check(lib.logismos_launch_window_attention_f32(P(qd), H * D, P(c.kp), P(c.vp), P(c.tables), P(keepd[0]), P(keepd[1]), P(out), H * D, T, c.mb, c.nb, H, G, D, C.byref(w),
                                                   P(st), stream()), "f32")
    want = np.concatenate([c.want(s, [p], host(qd).reshape(T, H, D)[i:i + 1], 0.2, size, keep, sink, gate[i:i + 1]) for i, (s, p) in enumerate(rows)])
    close(host(out).reshape(T, H, D), want, 3e-6)


# ---- gated linear attention ------------------------------------------------------------------------

def pad_heads(x, to):
    out = np.zeros(x.shape[:-1] + (to,))
    out[..., :x.shape[-1]] = x
    return out


def run_gla(form, heads, dk, dv, lens, seed, fp32=False, z_range=(-3.0, 6.0), tau=8.0):
    """Two calls over ragged sequences, the second continuing the first; outputs and states against the recurrence."""
    rng = np.random.default_rng(seed)
    pad = lambda d: max(32, 1 << (d - 1).bit_length())
    dp, wp, eps = pad(dk), pad(dv), 1e-5
    n, slots = len(lens), len(lens) + 2
    state, sl = fl(np.full((slots, heads, dp, wp), np.nan)), rng.permutation(slots)[:n]
    gain = rng.uniform(0.5, 1.5, (heads, dv))
    S = [np.zeros((heads, dk, dv)) for _ in lens]
    outs, wants = [], []
    for call in range(2):
        ll = lens if call == 0 else lens[::-1]
        T = sum(ll)
        q, k = rng.standard_normal((T, heads, dk)), rng.standard_normal((T, heads, dk))
        v, g = rng.standard_normal((T, heads, dv)), rng.standard_normal((T, heads, dv))
        z = rng.uniform(*z_range, (T, heads, dk))
        kw, vw = heads * dp, heads * wp
        proj = act(np.concatenate([pad_heads(q, dp).reshape(T, kw), pad_heads(k, dp).reshape(T, kw), pad_heads(v, wp).reshape(T, vw), pad_heads(g, wp).reshape(T, vw)], 1), fp32)
        ph = host(proj)
        cut = lambda at, h, d, p: ph[:, at:at + h * p].reshape(T, h, p)[..., :d]
        q, k, v, g = cut(0, heads, dk, dp), cut(kw, heads, dk, dp), cut(2 * kw, heads, dv, wp), cut(2 * kw + vw, heads, dv, wp)
        cu = np.concatenate([[0], np.cumsum(ll)])
        zd = np.zeros((T, heads, dp))
        rank, low, w2, w0 = 32, None, None, np.zeros((heads, dp))
        if form == "low":
            low = rng.standard_normal((T, rank))
            w2 = R.bf16(pad_heads(np.moveaxis(0.3 * rng.standard_normal((heads, dk, rank)), 1, 2), dp)).transpose(0, 2, 1).reshape(heads * dp, rank)
            w0[:, :dk] = rng.uniform(*z_range, (heads, dk))
            z = ((low.astype(np.float32).astype(np.float64) @ w2.T).reshape(T, heads, dp) + w0.astype(np.float32))[..., :dk]
        zd[..., :dk] = z
        out = act(np.zeros((T, vw + 8)), fp32)
        keep = [fl(zd.reshape(T, kw)) if low is None else None, None if low is None else fl(low), None if low is None else dev(w2, torch.bfloat16), fl(w0),
                fl(pad_heads(gain, wp)), ints(sl if call == 0 else sl[::-1]), torch.full((n,), 1 - call, dtype=torch.uint8, device=DEV), ints(cu)]
        a = TimeMix(A(proj), 2 * (kw + vw), 0, kw, 2 * kw, 2 * kw + vw, A(keep[0]), kw, A(keep[1]), rank, A(keep[2]), rank, rank, A(keep[3]), 0, A(keep[4]), A(state), A(keep[5]),
                    A(keep[6]), A(keep[7]), A(out), vw + 8, heads, dv, dp, 1.0, eps, 1, wp, tau, dk ** -0.5)
        if form == "chunked":
            check(lib.logismos_launch_time_mix_chunked_bf16(C.byref(a), n, stream()), "chunked")
        else:
            check(lib.logismos_launch_time_mix_step(C.byref(a), n, int(fp32), stream()), "step")
        alpha = np.exp(R.log_decay(z, tau))
        for i in range(n):
            s, r = (i if call == 0 else n - 1 - i), slice(cu[i], cu[i + 1])
            o = np.zeros((ll[i], heads, dv))
            for h in range(heads):
                o[:, h], S[s][h] = R.gla_recurrence(q[r, h] * dk ** -0.5, k[r, h], v[r, h], alpha[r, h], S[s][h])
            wants.append(R.rms_norm(o, gain, eps) * R.silu(g[r]))
        outs.append(host(out)[:, :vw].reshape(T, heads, wp))
    got, st = np.concatenate(outs), host(state)[sl]
    assert (got[..., dv:] == 0).all() and (st[:, :, dk:] == 0).all() and (st[..., dv:] == 0).all()
    return got[..., :dv], np.concatenate(wants), st[:, :, :dk, :dv], np.stack(S)


@pytest.mark.parametrize("heads,dk,dv", [(3, 24, 40), (2, 64, 64), (2, 128, 64), (1, 100, 128), (2, 20, 128), (2, 128, 20), (1, 130, 40), (1, 48, 200)])
@pytest.mark.parametrize("form", ["step", "low", "chunked"])
def test_gated_linear_attention(form, heads, dk, dv):
    if form == "chunked" and max(dk, dv) > 128:
        assert not lib.logismos_time_mix_has_chunked(max(64, 256 if dk > 128 else 64), 256 if dv > 128 else 64)
        return
    lens = [1, 1, 1] if form == "low" else [1, 2, 15, 16, 17, 63, 64, 65, 130]
    o, want, st, ends = run_gla(form, heads, dk, dv, lens, 3)
    close(o, want, 3e-3)
    close(st, ends, 3e-5)
    if form != "chunked":
        o, want, st, ends = run_gla(form, heads, dk, dv, lens, 4, fp32=True)
        close(o, want, 2e-5)
        close(st, ends, 3e-6)


@pytest.mark.parametrize("z_range,tau", [((-60.0, -20.0), 1.0), ((-200.0, 50.0), 1.0), ((5.0, 30.0), 16.0), ((-8.0, 0.0), 0.5)])
def test_strong_and_vanishing_decays(z_range, tau):
    """Decays that leave nothing of a state within a few tokens, and decays near one over a thousand."""
    for form in ("step", "chunked"):
        o, want, st, ends = run_gla(form, 2, 40, 24, [3, 70, 400], 5, z_range=z_range, tau=tau)
        close(o, want, 3e-3)
        close(st, ends, 3e-5)


# ---- mixtures of experts ---------------------------------------------------------------------------

MIXTURES = [(5, 2, 2, 2, 64, 128), (16, 4, 2, 1, 128, 256), (3, 0, 3, 0, 64, 64), (40, 3, 4, 1, 64, 192), (200, 100, 8, 0, 64, 64), (1, 0, 1, 3, 128, 128), (4, 300, 2, 1, 64, 64)]


def plain_mixture(h, z, corr, top, E, up, down, always):
    """Sum over the chosen experts and the ones that take every token; up [groups, 2, F, H], down [groups, H, F]."""
    chosen, weight = R.route(z, corr, top)
    out = np.zeros((h.shape[0], down.shape[1]))
    unit = lambda x, g: (R.silu(x @ up[g, 0].T) * (x @ up[g, 1].T)) @ down[g].T
    for e in range(z.shape[1]):
        t, s = np.nonzero(chosen == e)
        if t.size:
            out[t] += weight[t, s][:, None] * (unit(h[t], e) if e < E else h[t])
    for g in range(E, E + always):
        out += unit(h, g)
    return out


@pytest.mark.parametrize("E,I,top,always,F,H", MIXTURES)
@pytest.mark.parametrize("tokens,form", [(1, "few"), (7, "few"), (100, "few"), (130, "many"), (400, "many"), (33, "many"), (2500, "many"), (50, "f32"), (1, "router"), (9, "router"), (60, "router")])
def test_mixture_of_experts(E, I, top, always, F, H, tokens, form):
    if tokens > 1000 and E != 5:
        return
    rng = np.random.default_rng(E + tokens)
    n, G, pairs, fp32 = E + I, E + always, top + always, form == "f32"
    ld = -(-n // 16) * 16
    z, corr = np.zeros((tokens, ld)), 0.1 * rng.standard_normal(n)
    z[:, :n] = 2 * rng.standard_normal((tokens, n))
    if I == 300:
        corr[:E] -= 2.0       # every choice an identity expert: groups without rows
    z, corr = z.astype(np.float32), corr.astype(np.float32)
    wr = R.bf16(2 * rng.standard_normal((n, H)) / np.sqrt(H))
    hd = act(rng.standard_normal((tokens, H)), fp32)
    h = host(hd)
    if form == "router":      # the logits are a product of the rows: no close calls
        z[:, :n] = h @ wr.T
        ranked = -np.sort(-(R.softmax(z[:, :n].astype(np.float64)) + corr), axis=1)
        if top < n:
            corr = (corr + np.where((ranked[:, top - 1] - ranked[:, top]).min() < 1e-6, 1e-4 * rng.standard_normal(n), 0)).astype(np.float32)
    up = R.bf16(rng.standard_normal((G, 2, F, H)) / np.sqrt(H))
    down = R.bf16(rng.standard_normal((G, H, F)) / np.sqrt(F))
    wu = np.stack([np.concatenate([np.concatenate([up[g, 0, i:i + 32], up[g, 1, i:i + 32]]) for i in range(0, F, 32)]) for g in range(G)])
    keep = [fl(z), fl(corr), dev(wu, torch.bfloat16), dev(down, torch.bfloat16)]
    it = lambda *s: torch.full(s, -7, dtype=torch.int32, device=DEV)
    wts, prow, ident = fl(np.zeros((tokens, top))), it(tokens, pairs), fl(np.zeros(tokens))
    mid, rows = act(np.zeros((tokens * pairs, F)), fp32), act(np.full((tokens * pairs, H), np.nan), fp32)
    r = MoeRoute(A(keep[0]), ld, 1, A(keep[1]), E, I, top, always, A(wts), A(prow), A(ident))
    st, counts = status(), torch.zeros(E, dtype=torch.int32, device=DEV)
    if form != "many":
        off, tok = it(G + 1), it(tokens * pairs)
        r.offsets, r.row_token = A(off), A(tok)
        if form == "router":
            wrd, arrived = dev(wr, torch.bfloat16), torch.zeros(1, dtype=torch.int32, device=DEV)
            r.logits, r.h, r.w, r.width, r.arrived = 0, A(hd), A(wrd), H, A(arrived)
            check(lib.logismos_launch_moe_route(C.byref(r), tokens, stream()), "route")     # twice: it leaves its counter cleared
            assert not arrived.any()
        check(lib.logismos_launch_moe_route(C.byref(r), tokens, stream()), "route")
        if fp32:
            check(lib.logismos_launch_linear_experts_f32(P(hd), P(keep[2]), P(mid), P(off), P(tok), G, tokens, 2 * F, H, H, F, 4, 1.0, float("inf"), 0.0, stream()), "up")
            check(lib.logismos_launch_linear_experts_f32(P(mid), P(keep[3]), P(rows), P(off), P(None), G, tokens, H, F, F, H, 3, 0.0, 0.0, 0.0, stream()), "down")
        else:
            expected = -(-tokens * top // E)
            check(lib.logismos_launch_linear_experts_small_bf16(P(hd), P(keep[2]), P(mid), P(off), P(tok), G, tokens, expected, 2 * F, H, H, F, 2, 0, 0, 0, stream()), "up")
            check(lib.logismos_launch_linear_experts_small_bf16(P(mid), P(keep[3]), P(rows), P(off), P(None), G, tokens, expected, H, F, F, H, 0, 0, 0, 0, stream()), "down")
        o = off.cpu().numpy()
        assert o[0] == 0 and (np.diff(o) >= 0).all() and (np.diff(o)[E:] == tokens).all()
    else:
        mt = lib.logismos_moe_max_tiles(tokens, top, E, always)
        tiles, nt, pe, gat = it(mt, 4), it(1), it(tokens, top), act(np.zeros((tokens * pairs, H)), False)
        r.counts, r.pair_expert, r.tiles, r.n_tiles = A(counts), A(pe), A(tiles), A(nt)
        check(lib.logismos_launch_moe_route(C.byref(r), tokens, stream()), "route")
        check(lib.logismos_launch_moe_place(C.byref(r), P(hd), P(gat), H, tokens, stream()), "place")
        direct = always > 0
        check(lib.logismos_launch_linear_experts_tc_bf16(P(gat), tokens * pairs, P(hd if direct else None), tokens if direct else 0, P(keep[2]), P(mid), P(tiles), P(nt), mt, G, 2 * F,
                                                         H, H, F, 2, 0, 0, 0, P(st), stream()), "up")
        check(lib.logismos_launch_linear_experts_tc_bf16(P(mid), tokens * pairs, P(None), 0, P(keep[3]), P(rows), P(tiles), P(nt), mt, G, H, F, F, H, 0, 0, 0, 0, P(st), stream()), "down")
        assert nt.item() <= mt
    torch.cuda.synchronize()
    assert st.item() == 0
    # the choice itself: exact, and every pair has a row of its own
    chosen, weight = R.route(z[:, :n].astype(np.float64), corr.astype(np.float64), top)
    pr = prow.cpu().numpy()
    assert np.array_equal(pr[:, :top] < 0, chosen >= E) and (form == "router" or not keep[0][:, :n].any())
    close(host(wts), weight, 1e-5)
    close(host(ident) + 1e-3, np.where(chosen >= E, weight, 0).sum(1) + 1e-3, 1e-5)
    used = pr[pr >= 0]
    assert len(set(used)) == used.size and (used < tokens * pairs).all()
    # the sum, the norms around it and the residual
    x, one, zero = rng.standard_normal((tokens, H)), fl(np.ones(H)), fl(np.zeros(H))
    xd, post, nxt = fl(x), TanhNorm(0.1, A(one), A(zero)), TanhNorm(0.5, A(one), A(zero))
    m = MixtureOut(A(rows), A(prow), A(wts), A(ident), pairs, top, A(counts), E)
    check(lib.logismos_launch_tanh_norm(P(None), 0, C.byref(m), P(None), tokens, P(xd), C.byref(post), P(hd), C.byref(nxt), int(fp32), tokens, H, P(st), stream()), "sum")
    want = x + np.tanh(0.1 * plain_mixture(h, z[:, :n].astype(np.float64), corr.astype(np.float64), top, E, up, down, always))
    close(host(xd), want, 2e-6 if fp32 else 2e-3)
    close(host(hd), np.tanh(0.5 * want), 2e-6 if fp32 else 4e-3)
    assert not counts.any()


def test_equal_scores_choose_the_first_experts():
    z, n = fl(np.zeros((2, 16))), 7
    wts, prow, ident, off, tok = fl(np.zeros((2, 3))), torch.zeros((2, 3), dtype=torch.int32, device=DEV), fl(np.zeros(2)), ints(np.zeros(8)), ints(np.zeros(6))
    corr = fl(np.zeros(n))
    r = MoeRoute(A(z), 16, 0, A(corr), n, 0, 3, 0, A(wts), A(prow), A(ident), A(off), A(tok))
    check(lib.logismos_launch_moe_route(C.byref(r), 2, stream()), "route")
    assert off.tolist() == [0, 2, 4, 6, 6, 6, 6, 6] and np.allclose(host(wts), 1 / 3)


def test_grouped_projections_add_their_bias_to_the_main_columns():
    rng = np.random.default_rng(2)
    k, n_main, tail = 128, 256, 32
    w = R.bf16(rng.standard_normal((n_main + tail, k)) / np.sqrt(k))
    b = rng.standard_normal(n_main)
    for m, route in ((5, "small"), (200, "tc"), (20, "f32")):
        x = act(rng.standard_normal((m, k)), route == "f32")
        out, t = act(np.zeros((m, n_main)), route == "f32"), fl(np.zeros((m, tail)))
        wd, bd, st = dev(w, torch.bfloat16), fl(b), status()
        g = Groups(1, (i32 * 8)(n_main + tail), n_main, A(t), tail, 0.0, 0, A(bd))
        args = (P(x), P(wd), P(out), m, n_main + tail, k, k, n_main, C.byref(g))
        if route == "tc":
            check(lib.logismos_launch_linear_groups_tc_bf16(*args, P(st), stream()), route)
        else:
            check({"small": lib.logismos_launch_linear_groups_small_bf16, "f32": lib.logismos_launch_linear_groups_f32}[route](*args, stream()), route)
        want = host(x) @ w.T
        close(host(out), want[:, :n_main] + b, 1e-5 if route == "f32" else 3e-3)
        close(host(t), want[:, n_main:], 1e-5)


@pytest.mark.parametrize("m,n,k", [(1, 64, 64), (7, 192, 256), (16, 1024, 512), (12, 4096, 4096)])
@pytest.mark.parametrize("last", [False, True])
def test_output_projection_with_its_norms(m, n, k, last):
    rng = np.random.default_rng(n)
    ld = n + 64
    a, w = act(rng.standard_normal((m, k)), False), R.bf16(rng.standard_normal((n, k)) / np.sqrt(k))
    post, nxt, x = tanh_vectors(rng, n, ld), tanh_vectors(rng, n, ld), 2 * rng.standard_normal((m, ld))
    keep = [[fl(v) for v in p[1:]] for p in (post, nxt)]
    tp, tn = (TanhNorm(p[0], A(k_[0]), A(k_[1])) for p, k_ in zip((post, nxt), keep))
    xd, hd, wd = fl(x), act(np.zeros((m, ld)), False), dev(w, torch.bfloat16)
    check(lib.logismos_launch_linear_small_tanh_norm(P(a), P(wd), P(xd), C.byref(tp), P(hd), None if last else C.byref(tn), m, n, k, k, ld, stream()), "projection")
    want = x[:, :n] + R.tanh_norm(host(a) @ w.T, post[0], post[1][:n], post[2][:n])
    close(host(xd)[:, :n], want, 2e-6)
    assert np.array_equal(host(xd)[:, n:], x[:, n:].astype(np.float32)) and (host(hd)[:, n:] == 0).all()
    if last:
        assert not hd.any()
    else:
        close(host(hd)[:, :n], R.tanh_norm(want, nxt[0], nxt[1][:n], nxt[2][:n]), 3e-3)


@pytest.mark.parametrize("parts", [False, True])
def test_finishing_a_summed_projection(parts):
    rng = np.random.default_rng(3)
    m, n_main, tail = 50, 384, 32
    acc, b = rng.standard_normal((m, n_main + tail + 4)), rng.standard_normal(n_main)
    ad, bd, out, t = fl(acc), fl(b), act(np.zeros((m, n_main)), False), fl(np.zeros((m, tail)))
    tp = act(np.zeros((m, 2 * tail)), False) if parts else None
    g = Groups(1, (i32 * 8)(n_main + tail), n_main, A(t), tail, 2.0 if parts else 0.0, A(tp), A(bd))
    check(lib.logismos_launch_linear_groups_finish(P(ad), P(out), m, n_main + tail, n_main + tail + 4, n_main, C.byref(g), stream()), "finish")
    want = acc[:, n_main:n_main + tail]
    want = 2.0 * np.tanh(want / 2.0) if parts else want
    close(host(out), acc[:, :n_main] + b, 3e-3)
    close(host(t), want, 1e-6)
    assert not ad[:, :n_main + tail].any()
    if parts:
        close(host(tp)[:, :tail], want, 3e-3)
        close(host(tp)[:, :tail] + host(tp)[:, tail:], want, 2e-5)


@pytest.mark.parametrize("heads,rank,at,dims", [(3, 64, 24, 6), (16, 576, 512, 64), (20, 128, 40, 88), (40, 640, 8, 2), (64, 576, 512, 32)])
def test_latent_decode_turns_its_queries_and_gates_its_heads(heads, rank, at, dims):
    rng = np.random.default_rng(rank)
    lens = [1, 17, 64, 200]
    n, mb = len(lens), 14
    rot = {"dims": dims, "base": 500.0}
    nb = sum(-(-v // 16) for v in lens)
    tables, perm, used = -np.ones((n, mb), np.int32), rng.permutation(nb), 0
    pool = 0.5 * rng.standard_normal((nb, 16, rank))
    pd = act(pool, False)
    pool = host(pd)
    for s, v in enumerate(lens):
        b = -(-v // 16)
        tables[s, :b] = perm[used:used + b]
        used += b
    qd, gate = act(rng.standard_normal((n, heads, rank)), False), rng.standard_normal((n, heads + 3))
    q, gd, tab, td, cl = host(qd), fl(gate), angles(rot, 256), ints(tables), ints(lens)
    for chunk in (64, 1024):
        off = np.concatenate([[0], np.cumsum([-(-v // chunk) for v in lens])]).astype(np.int32)
        od, out, st = ints(off), act(np.zeros((n, heads, rank)), False), status()
        scr = torch.empty(lib.logismos_latent_decode_scratch_bytes(int(off[-1]), heads, rank), dtype=torch.uint8, device=DEV)
        check(lib.logismos_launch_latent_decode_bf16(P(qd), P(pd), P(td), P(cl), P(od), P(out), P(scr), n, int(off[-1]), chunk, mb, nb, heads, rank, 0.08, P(gd), heads + 3, P(tab), at,
                                                     dims, P(st), stream()), "decode")
        want = np.zeros((n, heads, rank))
        for s, v in enumerate(lens):
            c = pool[tables[s, np.arange(v) // 16], np.arange(v) % 16]
            x = q[s:s + 1].copy()
            x[..., at:at + dims] = R.rotate(x[..., at:at + dims], [v - 1], rot)
            for a in range(heads):
                want[s, a] = R.softmax(x[0, a] @ c.T * 0.08) @ c * R.sigmoid(gate[s, a])
        close(host(out), want, 8e-3)
        assert st.item() == 0


def test_launchers_reject_what_they_cannot_address():
    x, st = fl(np.zeros((4, 64))), status()
    one = fl(np.ones(64))
    t = TanhNorm(1.0, A(one), A(one))
    assert lib.logismos_launch_tanh_norm(P(x), 0, None, P(None), 4, P(x), None, P(x), None, 1, 4, 64, P(st), stream())          # neither norm
    assert lib.logismos_launch_tanh_norm(P(None), 0, None, P(None), 4, P(x), C.byref(t), P(x), None, 1, 4, 64, P(st), stream())  # nothing to add
    assert lib.logismos_launch_tanh_norm(P(x), 0, None, P(None), 4, P(x), None, P(x), C.byref(t), 1, 5, 64, P(st), stream())     # more rows than there are
    assert lib.logismos_launch_rotary_heads(P(x), 64, P(st), 1, 1, 64, 4, P(x), 8, 1, stream())                                   # part not at a multiple of eight
    w = Window(-1.0, 4, 0, 1, 0, 0)
    assert lib.logismos_launch_window_attention_f32(P(x), 64, P(x), P(x), P(st), P(st), P(st), P(x), 64, 1, 1, 1, 1, 1, 64, C.byref(w), P(st), stream())
    r = MoeRoute(A(x), 64, 0, A(x), 600, 0, 2, 0, A(x), A(x), A(x), A(x), A(x))
    assert lib.logismos_launch_moe_route(C.byref(r), 1, stream())
    torch.cuda.synchronize()
    assert st.item() == 0
