"""The kernels of the state-space / parallel decoder, each against the plain function of katadra_reference.py."""
import ctypes as C

import numpy as np
import pytest
import torch

import katadra_reference as R
from logismos_b200 import ops
from logismos_b200._lib import check, lib
from logismos_b200.structs import Groups, ScoreBias, Ssd, TimeMix

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
vp, i32, f32 = C.c_void_p, C.c_int32, C.c_float
P = lambda t: vp(0 if t is None else t.data_ptr())
A = lambda t: 0 if t is None else t.data_ptr()
stream = lambda: vp(torch.cuda.current_stream().cuda_stream)


def dev(a, dtype):
    return torch.from_numpy(np.ascontiguousarray(a)).to(DEV).to(dtype)


def fl(a):
    return dev(np.asarray(a, np.float32), torch.float32)


def ints(a):
    return dev(np.asarray(a, np.int32), torch.int32)


def close(got, want, tol):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    err = np.sqrt(np.mean((got - want) ** 2)) / np.sqrt(np.mean(want ** 2))
    assert err <= tol and np.abs(got - want).max() <= 12 * tol * np.abs(want).max(), (err, np.abs(got - want).max(), np.abs(want).max())


def pad_heads(x, dp):
    """[..., heads, d] -> [..., heads * dp] with zeros."""
    out = np.zeros(x.shape[:-1] + (dp,))
    out[..., :x.shape[-1]] = x
    return out.reshape(x.shape[:-2] + (-1,))


# ---- projections -----------------------------------------------------------------------------------

@pytest.mark.parametrize("m", [1, 7, 40, 300])
@pytest.mark.parametrize("route", ["tc", "small", "f32"])
def test_grouped_projections(m, route):
    """Blocks of columns with inputs of their own, bf16 columns and an fp32 tail with a soft cap."""
    rng = np.random.default_rng(m)
    k, ends, n_main, tail = 192, [256, 384, 640, 656], 640, 16
    w, a = R.bf16(rng.standard_normal((656, k)) / 14), R.bf16(rng.standard_normal((4, m, k)))
    t = torch.float32 if route == "f32" else torch.bfloat16
    wd, ad = dev(w, torch.bfloat16), dev(a, t)
    out, low = torch.full((m, n_main), 7.0, device=DEV, dtype=t), torch.full((m, tail + 4), 7.0, device=DEV)
    parts = torch.zeros((m, 2 * tail), device=DEV, dtype=torch.bfloat16)
    for cap in (0.0, 1.5):
        g = Groups(4, (i32 * 8)(*ends), n_main, A(low), tail + 4, cap, A(parts) if cap else 0)
        args = [P(ad), P(wd), P(out), m, 656, k, k, n_main, C.byref(g)]
        st = torch.zeros(1, dtype=torch.int32, device=DEV)
        fn = {"tc": lib.logismos_launch_linear_groups_tc_bf16, "small": lib.logismos_launch_linear_groups_small_bf16, "f32": lib.logismos_launch_linear_groups_f32}[route]
        check(fn(*args, *([P(st)] if route == "tc" else []), stream()), "groups")
        want = np.concatenate([a[i] @ w[b:e].T for i, (b, e) in enumerate(zip([0] + ends, ends))], axis=1)
        close(out.float().cpu(), want[:, :n_main], 1e-5 if route == "f32" else 3e-3)
        z = want[:, n_main:]
        close(low[:, :tail].cpu(), cap * np.tanh(z / cap) if cap else z, 1e-5)
        assert (low[:, tail:] == 7.0).all() and int(st) == 0
        if cap and route != "f32":
            assert (parts[:, :tail].double() + parts[:, tail:].double() - low[:, :tail].double()).abs().max() <= 2 ** -16 * low[:, :tail].abs().max()
    bad = Groups(4, (i32 * 8)(100, 384, 640, 656), n_main, A(low), tail + 4, 0.0)
    assert lib.logismos_launch_linear_groups_small_bf16(P(ad), P(wd), P(out), m, 656, k, k, n_main, C.byref(bad), stream()) == 1


@pytest.mark.parametrize("m", [3, 90])
def test_squared_relu_epilogue(m):
    rng = np.random.default_rng(1)
    a, w = R.bf16(rng.standard_normal((m, 128))), R.bf16(rng.standard_normal((192, 128)) / 11)
    want = np.maximum(a @ w.T, 0) ** 2
    ad, wd, out = dev(a, torch.bfloat16), dev(w, torch.bfloat16), torch.zeros((m, 192), device=DEV, dtype=torch.bfloat16)
    st = torch.zeros(1, dtype=torch.int32, device=DEV)
    check(lib.logismos_launch_linear_small_bf16(P(ad), P(wd), P(None), P(out), m, 192, 128, 128, 192, 1, 0, 0, 0, 5, 0, 0, 0, stream()), "small")
    close(out.float().cpu(), want, 3e-3)
    out.zero_()
    check(lib.logismos_launch_linear_t_act_bf16(P(ad), P(wd), P(None), P(out), m, 192, 128, 128, 192, 5, 0, 0, 0, P(st), stream()), "tc")
    close(out.float().cpu(), want, 3e-3)
    af, of = fl(a), torch.zeros((m, 192), device=DEV)
    check(lib.logismos_launch_linear_f32(P(af), P(wd), P(None), P(of), m, 192, 128, 128, 192, 1, 0, 0, 0, 5, 0, 0, 0, stream()), "f32")
    close(of.cpu(), want, 1e-5)


# ---- norm and token shift --------------------------------------------------------------------------

@pytest.mark.parametrize("n,ld", [(40, 64), (130, 192), (2050, 2112), (5000, 5056)])
@pytest.mark.parametrize("out32", [0, 1])
def test_output_norm_and_shift(n, ld, out32):
    rng = np.random.default_rng(n)
    T, eps = 9, 1e-3
    pad = lambda a: np.pad(a, [(0, 0)] * (a.ndim - 1) + [(0, ld - n)])
    y, x, w, b, mu = rng.standard_normal((T, n)) + 3, rng.standard_normal((T, n)), 1 + 0.3 * rng.standard_normal(n), rng.standard_normal(n), rng.standard_normal((5, n))
    want = x + R.layer_norm(y, w, b, eps)
    yd, xd, wd, bd, md = (fl(pad(v)) for v in (y, x, w, b, mu))
    odt, tol = (torch.float32, 1e-6) if out32 else (torch.bfloat16, 3e-3)
    h = torch.zeros((6, T, ld), device=DEV, dtype=odt)
    check(lib.logismos_launch_post_norm(P(yd), 1, P(None), T, P(xd), P(wd), P(bd), P(h), out32, T, n, ld, eps, P(None), stream()), "norm")
    close(xd.cpu()[:, :n], want, 1e-6)
    close(h[0].float().cpu()[:, :n], want, tol)
    assert (xd[:, n:] == 0).all() and (yd == 0).all()
    # gathered rows without a residual
    rows = ints([8, 0, 8])
    check(lib.logismos_launch_post_norm(P(xd), 0, P(rows), T, P(None), P(wd), P(bd), P(h), out32, 3, n, ld, eps, P(None), stream()), "norm")
    close(h[0, :3].float().cpu()[:, :n], R.layer_norm(want, w, b, eps)[[8, 0, 8]], tol)
    # mixes of ragged sequences: 4 tokens that continue slot 2, one that starts slot 0, 4 that start slot 1
    state = fl(rng.standard_normal((3, 2, ld)))
    state[..., n:] = 0
    before = state.cpu().numpy().astype(np.float64)
    cu, seq, slots = ints([0, 4, 5, 9]), ints([0] * 4 + [1] + [2] * 4), ints([2, 0, 1])
    fresh, phase = dev(np.array([0, 1, 1], np.uint8), torch.uint8), dev(np.array([1, 0, 1], np.uint8), torch.uint8)
    check(lib.logismos_launch_token_shift(P(xd), P(h), out32, P(md), 5, P(state), P(slots), P(fresh), P(phase), P(seq), P(cu), T, ld, stream()), "shift")
    prev = np.concatenate([before[2, 1, :n][None], want[:3], np.zeros((1, n)), np.zeros((1, n)), want[5:8]])
    got = h.float().cpu().numpy()
    close(got[0][:, :n], want, tol)
    for s in range(5):
        close(got[s + 1][:, :n], want + (prev - want) * mu[s], tol)
    after = state.cpu().numpy()
    for k, (sl, ph, last) in enumerate(((2, 1, 3), (0, 0, 4), (1, 1, 8))):
        close(after[sl, 1 - ph, :n], want[last], 1e-6)
        assert np.array_equal(after[sl, ph], before[sl, ph].astype(np.float32))
    # one token per sequence in one launch
    yd, xd = fl(pad(y)), fl(pad(x))
    check(lib.logismos_launch_post_norm_shift_decode(P(yd), 0, P(xd), P(wd), P(bd), P(h), out32, P(md), 5, P(state), P(slots), P(fresh), P(phase), 3, n, ld, eps, stream()), "decode")
    got = h.reshape(-1)[:6 * 3 * ld].reshape(6, 3, ld).float().cpu().numpy()
    prev = np.stack([before[2, 1, :n], np.zeros(n), np.zeros(n)])
    for s in range(6):
        close(got[s][:, :n], want[:3] + ((prev - want[:3]) * mu[s - 1] if s else 0), tol)
    close(state.cpu().numpy()[2, 0, :n], want[0], 1e-6)


# ---- time mixing -----------------------------------------------------------------------------------

def run_time_mix(form, heads, d, lens, seed, fp32=False, z_lo=-6.0, z_hi=1.0, split_at=None):
    """Sequences of `lens` tokens (the last continues a given state); returns outputs, reference, states, reference states."""
    rng = np.random.default_rng(seed)
    dp = next(p for p in (32, 64, 128, 256) if p >= d)
    T, rank, eps, scale = sum(lens), 64, 1e-5, 0.7
    rnd = (lambda a: a) if fp32 else R.bf16
    r, k, v, g = (rnd(rng.standard_normal((T, heads, d))) for _ in range(4))
    low, w2 = np.tanh(rng.standard_normal((T, 40))), R.bf16(rng.standard_normal((heads, d, 40)) / 12)
    w0, u, gain = rng.uniform(z_lo, z_hi, (heads, d)), rng.standard_normal((heads, d)), 1 + 0.3 * rng.standard_normal((heads, d))
    w0, u, gain = (a.astype(np.float32).astype(np.float64) for a in (w0, u, gain))
    low = low.astype(np.float32).astype(np.float64)
    z = np.einsum("tr,hdr->thd", low, w2) + w0
    S0 = rng.standard_normal((len(lens), heads, d, d))
    want, ends, at = [], [], 0
    for s, n in enumerate(lens):
        o, e = zip(*[R.time_mix_recurrence(r[at:at + n, h], k[at:at + n, h], v[at:at + n, h], np.exp(-np.exp(z[at:at + n, h])), u[h],
                                           S0[s, h] if s == len(lens) - 1 else None) for h in range(heads)])
        o = np.stack(o, axis=1)
        want.append((R.unit_rms(o, eps) * gain * R.silu(g[at:at + n]) * scale))
        ends.append(np.stack(e))
        at += n
    odt = torch.float32 if fp32 else torch.bfloat16
    proj = dev(np.concatenate([pad_heads(a, dp) for a in (r, k, v, g)], axis=1), odt)
    W = heads * dp
    w2p = np.zeros((heads, dp, 2 * rank))
    w2p[:, :d, :40], w2p[:, :d, rank:rank + 40] = w2, w2
    lowd = fl(np.pad(low, [(0, 0), (0, rank - 40)]))
    zd = fl(pad_heads(z, dp)) if form != "low" else None
    if zd is not None:
        zd.reshape(T, heads, dp)[..., d:] = 0.3
    state = torch.full((len(lens) + 1, heads, dp, dp), 9.0, device=DEV)
    slots = [len(lens) - i for i in range(len(lens))]
    full = np.zeros((heads, dp, dp))
    full[:, :d, :d] = S0[-1]
    state[slots[-1]] = fl(full)
    fresh = np.ones(len(lens), np.uint8)
    fresh[-1] = 0
    out = torch.full((T, W + 16), 5.0, device=DEV, dtype=odt)
    keep = [proj, zd, lowd, dev(w2p.reshape(W, -1), torch.bfloat16), fl(pad_heads(w0, dp)), fl(pad_heads(u, dp)), fl(pad_heads(gain, dp)), state, ints(slots),
            dev(fresh, torch.uint8), ints(np.concatenate([[0], np.cumsum(lens)])), out]
    a = TimeMix(A(proj), 4 * W, 0, W, 2 * W, 3 * W, A(zd), W, A(lowd), rank, A(keep[3]), 2 * rank, rank, A(keep[4]), A(keep[5]), A(keep[6]), A(state), A(keep[8]),
                A(keep[9]), A(keep[10]), A(out), W + 16, heads, d, dp, scale, eps)
    if form == "chunked":
        check(lib.logismos_launch_time_mix_chunked_bf16(C.byref(a), len(lens), stream()), "chunked")
    else:
        check(lib.logismos_launch_time_mix_step(C.byref(a), len(lens), int(fp32), stream()), "step")
    torch.cuda.synchronize()
    o = out.float().cpu().numpy()
    assert (o[:, W:] == 5.0).all()
    o = o[:, :W].reshape(T, heads, dp)
    assert (o[..., d:] == 0).all() and (state[0] == 9.0).all()
    st = state.cpu().numpy()[slots]
    assert (st[:, :, d:] == 0).all() and (st[..., d:] == 0).all()
    return o[..., :d], np.concatenate(want), st[:, :, :d, :d], np.stack(ends)


@pytest.mark.parametrize("heads,d", [(3, 24), (2, 64), (1, 100), (2, 130)])
@pytest.mark.parametrize("form", ["step", "low", "chunked"])
def test_time_mixing(form, heads, d):
    if form == "chunked" and d > 128:
        assert not lib.logismos_time_mix_has_chunked(256, 256)
        return
    lens = [1, 1, 1] if form == "low" else [1, 2, 15, 16, 17, 63, 64, 65, 130]
    o, want, st, ends = run_time_mix(form, heads, d, lens, 3)
    close(o, want, 3e-3)
    close(st, ends, 3e-5)
    if form != "chunked":
        o, want, st, ends = run_time_mix(form, heads, d, lens, 4, fp32=True)
        close(o, want, 3e-6)
        close(st, ends, 2e-6)


@pytest.mark.parametrize("z_lo,z_hi", [(-9.0, -5.0), (1.0, 2.2), (-6.0, 4.0), (3.0, 6.0)])
def test_chunked_time_mixing_over_the_range_of_decays(z_lo, z_hi):
    """From hardly any decay to a state that is gone within a token, where block products would overflow."""
    o, want, st, ends = run_time_mix("chunked", 2, 64, [64, 33, 150], 5, z_lo=z_lo, z_hi=z_hi)
    close(o, want, 4e-3)
    close(st, ends, 5e-5)


# ---- state-space mixer -----------------------------------------------------------------------------

def run_ssd(form, heads, v, groups, n, taps, lens, seed, fp32=False, a_hi=1.0):
    rng = np.random.default_rng(seed)
    pow2 = lambda x, lo: next(p for p in (16, 32, 64, 128, 256) if p >= max(x, lo))
    V, N = pow2(v, 16), pow2(n, 32)
    T, inner, ch, pch = sum(lens), heads * v, heads * v + 2 * groups * n, heads * V + 2 * groups * N
    rnd = (lambda a: a.astype(np.float32).astype(np.float64)) if fp32 else R.bf16
    raw, dt = rnd(rng.standard_normal((T, ch))), rng.standard_normal((T, heads)).astype(np.float32).astype(np.float64)
    cw, cb = (rng.standard_normal((ch, taps)) / np.sqrt(taps)).astype(np.float32).astype(np.float64), 0.2 * rng.standard_normal(ch).astype(np.float32).astype(np.float64)
    dtb, la, D = (x.astype(np.float32).astype(np.float64) for x in (rng.uniform(-4, 1, heads), rng.uniform(-2, a_hi, heads), rng.standard_normal(heads)))
    S0, past = rng.standard_normal((heads, n, v)), rnd(rng.standard_normal((taps - 1, ch)))
    want, ends, at = [], [], 0
    for s, m in enumerate(lens):
        last = s == len(lens) - 1
        x = np.concatenate([past if last else np.zeros((taps - 1, ch)), raw[at:at + m]])
        xbc = R.silu(R.causal_conv(x, cw, cb))[taps - 1:]
        if not fp32:
            xbc = R.bf16(xbc)
        xx, B, Cc = xbc[:, :inner].reshape(m, heads, v), xbc[:, inner:inner + groups * n].reshape(m, groups, n), xbc[:, inner + groups * n:].reshape(m, groups, n)
        y, e = zip(*[R.ssd_recurrence(xx[:, h], B[:, h // (heads // groups)], Cc[:, h // (heads // groups)], R.softplus(dt[at:at + m, h] + dtb[h]), la[h], D[h],
                                      S0[h] if last else None) for h in range(heads)])
        want.append(np.stack(y, axis=1))
        ends.append((np.stack(e), x[m:]))
        at += m

    def chan(a):  # channel layout with padding, last axis
        return np.concatenate([pad_heads(a[..., :inner].reshape(a.shape[:-1] + (heads, v)), V), pad_heads(a[..., inner:].reshape(a.shape[:-1] + (2 * groups, n)), N)], axis=-1)

    odt = torch.float32 if fp32 else torch.bfloat16
    proj = dev(np.concatenate([np.zeros((T, heads * V)), chan(raw)], axis=1), odt)
    k = len(lens)
    slots = [k - i for i in range(k)]
    state, cstate = torch.full((k + 1, heads, N, V), 9.0, device=DEV), torch.full((k + 1, 2, max(taps - 1, 1), pch), 9.0, device=DEV)
    full = np.zeros((heads, N, V))
    full[:, :n, :v] = S0
    state[slots[-1]] = fl(full)
    phase = rng.integers(0, 2, k)
    if taps > 1:
        cstate[slots[-1], int(phase[-1])] = fl(chan(past))
    fresh = np.ones(k, np.uint8)
    fresh[-1] = 0
    y, xbc_d = torch.full((T, heads * V), 5.0, device=DEV, dtype=odt), torch.zeros((T, pch), device=DEV, dtype=odt)
    cu, seq = ints(np.concatenate([[0], np.cumsum(lens)])), ints(np.repeat(np.arange(k), lens))
    keep = [fl(dt), fl(np.ascontiguousarray(chan(cw.T))), fl(chan(cb)), fl(dtb), fl(la), fl(D), ints(slots), dev(fresh, torch.uint8), dev(phase.astype(np.uint8), torch.uint8), cu]
    a = Ssd(A(proj), proj.shape[1], A(keep[0]), heads, A(keep[1]), A(keep[2]), A(cstate), taps, A(keep[3]), A(keep[4]), A(keep[5]), A(state), A(keep[6]), A(keep[7]),
            A(keep[8]), A(cu), A(y), heads * V, heads, groups, N, V, A(xbc_d), pch)
    single = all(m == 1 for m in lens)
    check(lib.logismos_launch_ssd_conv(C.byref(a), P(seq), 0, T, int(single), int(fp32), stream()), "conv")
    if form == "chunked":
        check(lib.logismos_launch_ssd_chunked_bf16(C.byref(a), k, stream()), "chunked")
    elif form == "segments":
        entries = T // 256 + k + 1
        scr = torch.full((lib.logismos_ssd_scratch_bytes(entries, heads, N, V) // 4,), float("nan"), device=DEV)
        check(lib.logismos_launch_ssd_segmented_bf16(C.byref(a), k, max(lens), P(scr), entries, stream()), "segments")
    else:
        check(lib.logismos_launch_ssd_step(C.byref(a), k, int(fp32), stream()), "step")
    torch.cuda.synchronize()
    got = y.float().cpu().numpy().reshape(T, heads, V)
    assert (got[..., v:] == 0).all() and (state[0] == 9.0).all() and (cstate[0] == 9.0).all()
    st = state.cpu().numpy()[slots]
    assert (st[:, :, n:] == 0).all() and (st[..., v:] == 0).all()
    if taps > 1:
        for s in range(k):
            assert np.allclose(cstate[slots[s], 1 - int(phase[s])].cpu().numpy(), chan(ends[s][1]), rtol=0, atol=1e-6), s
        assert np.array_equal(cstate[slots[-1], int(phase[-1])].cpu().numpy(), chan(past).astype(np.float32))
    return got[..., :v], np.concatenate(want), st[:, :, :n, :v], np.stack([e[0] for e in ends])


@pytest.mark.parametrize("heads,v,groups,n,taps", [(6, 12, 2, 20, 4), (4, 64, 1, 128, 4), (2, 16, 1, 30, 2)])
def test_state_space_recurrence_in_segments(heads, v, groups, n, taps):
    """Decays that depend on the data, over segments that run side by side."""
    for lens in ([1200], [256, 257, 3, 600]):
        o, want, st, ends = run_ssd("segments", heads, v, groups, n, taps, lens, 7)
        close(o, want, 4e-3)
        close(st, ends, 3e-3)


@pytest.mark.parametrize("heads,v,groups,n,taps", [(6, 12, 2, 20, 4), (4, 64, 1, 128, 4), (2, 100, 2, 60, 1), (3, 20, 3, 100, 8), (2, 16, 1, 30, 2), (2, 140, 1, 70, 3), (1, 40, 1, 200, 3)])
@pytest.mark.parametrize("form", ["step", "chunked"])
def test_state_space_recurrence(form, heads, v, groups, n, taps):
    if form == "chunked" and (v > 128 or n > 128):
        assert not lib.logismos_ssd_has_chunked(256, 64) and not lib.logismos_ssd_has_chunked(64, 256)
        return
    lens = [1, 2, 3, 5, 16, 17, 63, 64, 65, 2 if heads == 6 else 140]
    o, want, st, ends = run_ssd(form, heads, v, groups, n, taps, lens, 7)
    close(o, want, 4e-3)
    close(st, ends, 3e-3)   # a convolved input on a rounding border moves the state by half a unit
    if form == "step":
        o, want, st, ends = run_ssd(form, heads, v, groups, n, taps, [1] * 5, 9)
        close(o, want, 4e-3)
        o, want, st, ends = run_ssd(form, heads, v, groups, n, taps, lens, 8, fp32=True)
        close(o, want, 3e-6)
        close(st, ends, 3e-6)


def test_state_space_with_fast_decay():
    o, want, st, ends = run_ssd("chunked", 4, 64, 2, 64, 4, [64, 200], 9, a_hi=5.0)
    close(o, want, 4e-3)


@pytest.mark.parametrize("heads,v,parts", [(4, 32, 2), (6, 24, 3), (5, 12, 4), (8, 64, 8), (3, 40, 1), (64, 64, 1), (130, 128, 1)])
@pytest.mark.parametrize("fp32", [False, True])
def test_gate_and_norm_in_parts(heads, v, parts, fp32):
    rng = np.random.default_rng(heads)
    V, T = next(p for p in (16, 32, 64, 128, 256) if p >= v), 5
    rnd = (lambda a: a) if fp32 else R.bf16
    y, z, gain = rnd(rng.standard_normal((T, heads, v))), rnd(rng.standard_normal((T, heads, v))), 1 + 0.3 * rng.standard_normal((heads, v))
    want = R.grouped_unit_rms((y * R.silu(z)).reshape(T, -1), parts, 0.01) * gain.reshape(-1)
    odt = torch.float32 if fp32 else torch.bfloat16
    yd, zd, gd = dev(pad_heads(y, V), odt), dev(np.pad(pad_heads(z, V), [(0, 0), (0, 24)]), odt), fl(pad_heads(gain, V))
    out = torch.zeros((T, heads * V + 8), device=DEV, dtype=odt)
    check(lib.logismos_launch_gated_group_norm(P(yd), heads * V, P(zd), heads * V + 24, P(gd), P(out), heads * V + 8, int(fp32), T, heads, v, V, parts, 0.01, stream()), "norm")
    got = out.float().cpu().numpy()[:, :heads * V].reshape(T, heads, V)[..., :v].reshape(T, -1)
    close(got, want, 2e-6 if fp32 else 3e-3)


# ---- attention -------------------------------------------------------------------------------------

def bias_table(rel, far):
    """The kernels' table: by head and distance up to `far`, in units of log2."""
    rows = [R.distance_bucket(n, rel.shape[0], far) for n in range(far + 1)]
    return fl(np.ascontiguousarray(rel[rows].T) / np.log(2.0))


def query_bound(n, coef, every):
    return 1.02 * max(R.query_temperature(p, coef, every) for p in range(n))


def attention_case(H, G, dim, vdim, lens, new, far, cap, rel_rows=9, seed=0, coef=0.5, every=10.0, fp32=False, scale=None, stand_out=True, bounded_qk=True):
    """Sequences with lens[i] keys of which the last new[i] are this step's; every new row's output."""
    rng = np.random.default_rng(seed)
    D = next(p for p in (64, 128, 256) if p >= max(dim, vdim))
    rnd = (lambda a: a.astype(np.float32).astype(np.float64)) if fp32 else R.bf16
    eps, gscale, scale = 1e-4, 0.6, scale or 2.0 / np.sqrt(dim)
    rel = 2.0 * rng.standard_normal((rel_rows, H))
    nb = sum(-(-n // 16) for n in lens) + 3
    perm, at = rng.permutation(nb), 0
    tables = -np.ones((len(lens), max(-(-n // 16) for n in lens) + 1), np.int32)
    odt = torch.float32 if fp32 else torch.bfloat16
    kp, vpool = (torch.full((nb, 16, G * D), 3.0, device=DEV, dtype=odt) for _ in range(2))
    ld = (2 * H + 2 * G) * D
    rows, pos, slots, want, cached, gates = [], [], [], [], [], []
    for s, n in enumerate(lens):
        m = -(-n // 16)
        tables[s, :m] = perm[at:at + m]
        at += m
        q, k, v, g = rnd(rng.standard_normal((n, H, dim))), rnd(rng.standard_normal((n, G, dim))), rnd(rng.standard_normal((n, G, vdim))), rnd(rng.standard_normal((n, H, vdim)))
        if stand_out and n > 4:   # the last query finds one key far away
            q[-1] = k[1, np.arange(H) // (H // G)]
            v[1] *= 8
        p0 = n - new[s]
        qn, kn = R.unit_rms(q, eps), R.unit_rms(k, eps)
        qn = qn * np.array([R.query_temperature(p, coef, every) for p in range(n)])[:, None, None]
        o = np.zeros((n, H, vdim))
        bias = rel[[R.distance_bucket(d, rel_rows, far) for d in range(n)]]
        for h in range(H):
            sc = R.attention_scores(qn[:, h], kn[:, h // (H // G)], scale, cap, bias[:, h]) if cap else np.where(
                np.tri(n) > 0, qn[:, h] @ kn[:, h // (H // G)].T * scale + bias[np.maximum(np.arange(n)[:, None] - np.arange(n), 0), h], -np.inf)
            o[:, h] = R.softmax(sc) @ v[:, h // (H // G)]
        want.append((o * R.sigmoid(g) * gscale)[p0:])
        rows.append(np.concatenate([pad_heads(a, D) for a in (q, k, v, g)], axis=1))
        pos.append(np.arange(n)); slots.append(tables[s, np.arange(n) // 16].astype(np.int64) * 16 + np.arange(n) % 16)
        cached.append(p0)
    # all rows go through the unit-and-store kernel; only the new ones attend
    allrows, allpos, allslots = dev(np.concatenate(rows), odt), ints(np.concatenate(pos)), dev(np.concatenate(slots), torch.int64)
    st = torch.zeros(1, dtype=torch.int32, device=DEV)
    T = sum(lens)
    check(lib.logismos_launch_unit_qk_store(P(allrows), ld, P(kp), P(vpool), P(allslots), P(allpos), T, H, G, D, dim, eps, coef, every, nb * 16, int(fp32), P(st), stream()), "unit")
    sel = np.concatenate([np.arange(a + c, a + n) for a, n, c in zip(np.concatenate([[0], np.cumsum(lens)[:-1]]), lens, cached)])
    q = allrows[torch.from_numpy(sel).to(DEV)].contiguous()
    table, mb = bias_table(rel, far), tables.shape[1]
    hot = dim * query_bound(max(lens), coef, every) if bounded_qk else 0.0
    sb = ScoreBias(scale, cap, A(table), far, float(np.abs(rel).max()), hot, A(q) + (H + 2 * G) * D * (4 if fp32 else 2), ld, gscale)
    out, td = torch.full((len(sel), H * D + 8), 5.0, device=DEV, dtype=odt), ints(tables)
    if fp32:
        sid, ps = ints(np.repeat(np.arange(len(lens)), new)), ints(np.concatenate([np.arange(c, n) for c, n in zip(cached, lens)]))
        check(lib.logismos_launch_bias_attention_f32(P(q), ld, P(kp), P(vpool), P(td), P(sid), P(ps), P(out), H * D + 8, len(sel), mb, nb, H, G, D, C.byref(sb), P(st), stream()), "f32")
    elif max(new) == 1:
        cl = torch.tensor(lens, dtype=torch.int32)
        off, total = ops.build_decode_chunks(cl, 64)
        scr = torch.empty(lib.logismos_paged_decode_scratch_bytes(total, H, D), dtype=torch.uint8, device=DEV)
        cd, od = cl.to(DEV), off.to(DEV)
        check(lib.logismos_launch_bias_attention_decode_bf16(P(q), ld, P(kp), P(vpool), P(td), P(cd), P(od), P(out), H * D + 8, P(scr), len(lens), total, 64, mb, nb, H, G, D,
                                                             C.byref(sb), P(st), stream()), "decode")
    else:
        scr = torch.empty(lib.logismos_paged_prefix_attention_scratch_bytes(T, len(lens), G, D), dtype=torch.uint8, device=DEV)
        cu, kv = ints(np.concatenate([[0], np.cumsum(new)])), ints(lens)
        check(lib.logismos_launch_bias_attention_prefix_bf16(P(q), ld, P(cu), P(kv), P(kp), P(vpool), P(td), mb, nb, P(out), H * D + 8, P(scr), len(sel), T, len(lens), max(new),
                                                             max(lens), H, G, D, C.byref(sb), P(st), stream()), "prefix")
    torch.cuda.synchronize()
    assert int(st) == 0 and (out[:, H * D:] == 5.0).all()
    got = out.float().cpu().numpy()[:, :H * D].reshape(len(sel), H, D)
    assert (got[..., vdim:] == 0).all()
    return got[..., :vdim], np.concatenate(want)


SHAPES = [(4, 4, 48, 64, 240, 30.0), (6, 2, 24, 40, 33, 4.0), (20, 1, 64, 16, 7, 30.0), (2, 1, 128, 100, 150, 12.0), (2, 2, 200, 256, 20, 25.0)]


@pytest.mark.parametrize("H,G,dim,vdim,far,cap", SHAPES)
def test_decode_attention(H, G, dim, vdim, far, cap):
    lens = [1, 2, far, far + 1, far + 2, 16, 17, 64, 65, 300]
    got, want = attention_case(H, G, dim, vdim, lens, [1] * len(lens), far, cap)
    close(got, want, 6e-3)


@pytest.mark.parametrize("H,G,dim,vdim,far,cap", SHAPES)
def test_prompt_attention(H, G, dim, vdim, far, cap):
    """Whole prompts and continuations, keys near and far from every tile border; capped scores that need no
    running maximum and (a cap or bias too large for that) scores that do."""
    lens, new = [2, 130, 129, 300, 260], [2, 130, 5, 300, 128]
    for bounded in (True, False):     # the cap as a polynomial where q . k is known to be small enough, else by exponentials
        got, want = attention_case(H, G, dim, vdim, lens, new, far, cap, seed=1, bounded_qk=bounded)
        close(got, want, 6e-3)
    got, want = attention_case(H, G, dim, vdim, lens, new, far, 30.0, seed=1, scale=0.1 / np.sqrt(dim), coef=0.2, every=500.0)
    close(got, want, 6e-3)
    got, want = attention_case(H, G, dim, vdim, [200, 140], [200, 7], far, 90.0, seed=2)
    close(got, want, 6e-3)
    got, want = attention_case(H, G, dim, vdim, [200, 140], [200, 7], far, 0.0, seed=3, coef=0.0)
    close(got, want, 6e-3)


@pytest.mark.parametrize("H,G,dim,vdim,far,cap", SHAPES)
def test_fp32_attention(H, G, dim, vdim, far, cap):
    got, want = attention_case(H, G, dim, vdim, [1, 40, 200], [1, 40, 3], far, cap, seed=4, fp32=True)
    close(got, want, 3e-6)


def test_bias_table_edges_show():
    """Distances on both sides of every bucket border: a table that is one off moves the output."""
    rng = np.random.default_rng(0)
    rel_rows, far = 8, 50
    borders = [n for n in range(1, far + 2) if R.distance_bucket(n, rel_rows, far) != R.distance_bucket(n - 1, rel_rows, far)]
    assert len(borders) == rel_rows - 1 and borders[:4] == [1, 2, 3, 4]
    rel = 6.0 * rng.standard_normal((rel_rows, 1))
    want = bias_table(rel, far)[0].cpu().numpy()
    for b in borders:
        assert abs(want[b] - want[b - 1]) > 1e-3
    got, ref = attention_case(2, 1, 16, 16, borders + [b + 1 for b in borders], [1] * (2 * len(borders)), far, 20.0, rel_rows=rel_rows, seed=5, scale=0.3, stand_out=False)
    close(got, ref, 6e-3)
