"""Every kernel of the latent-attention decoder alone, against the plain functions of latent_reference.py
(float64) on the same bf16 or fp32 inputs."""
import numpy as np
import pytest
import torch

import latent_reference as R
from gpu_util import DEV, TOL, bf16_cuda, row_rel, to_np
from logismos_b200 import ops

pytestmark = pytest.mark.gpu
F32 = 3e-6


def f32(x):
    return torch.from_numpy(np.ascontiguousarray(x, dtype=np.float32)).to(DEV)


def i32(x):
    return torch.from_numpy(np.ascontiguousarray(x, dtype=np.int32)).to(DEV)


def u8(x):
    return torch.from_numpy(np.ascontiguousarray(x, dtype=np.uint8)).to(DEV)


def interleave(g, u):
    """Gate and up rows in blocks of 32, the order of the gated epilogues."""
    n = g.shape[0] // 32
    return np.concatenate([np.stack([g.reshape(n, 32, -1)[i], u.reshape(n, 32, -1)[i]]).reshape(64, -1) for i in range(n)])


@pytest.mark.parametrize("route", ["small", "tcgen05", "f32"])
@pytest.mark.parametrize("m,n,k", [(1, 16, 64), (7, 48, 192), (9, 330, 128), (33, 64, 1088), (64, 400, 320), (65, 1040, 4160), (130, 4816, 64)])
def test_linear_epilogues(route, m, n, k):
    rng = np.random.default_rng(m * n + k)
    at, a = bf16_cuda(rng.standard_normal((m, k)))
    wt, w = bf16_cuda(rng.standard_normal((n, k)) / np.sqrt(k))
    b = rng.standard_normal(n).astype(np.float32)
    if route == "f32":
        at, a = f32(rng.standard_normal((m, k))), None
        a = at.cpu().numpy()
    kw = dict(small=route == "small")
    z = a.astype(np.float64) @ w.astype(np.float64).T + b
    tol = F32 * 4 if route == "f32" else 2e-5
    got = to_np(ops.linear_act(at, wt, f32(b), ops.EPI_F32, (1.5, 0.0, 0.0), **kw))
    assert np.abs(got - R.softcap(z, 1.5)).max() <= tol * 10
    got = to_np(ops.linear_act(at, wt, None, ops.EPI_F32, **kw))
    assert np.abs(got - (z - b)).max() <= tol * max(1.0, np.abs(z).max())
    if n % 16 == 0:
        if route != "f32":
            assert row_rel(to_np(ops.linear_act(at, wt, f32(b), ops.EPI_BF16, **kw)), z) <= 6e-3
        x0 = rng.standard_normal((m, n)).astype(np.float32)
        x = f32(x0)
        ops.linear_act(at, wt, f32(b), residual=x, **kw)
        assert np.abs(to_np(x) - (x0 + z)).max() <= tol * max(1.0, np.abs(z).max())


@pytest.mark.parametrize("route", ["small", "tcgen05", "f32"])
@pytest.mark.parametrize("m,ff,k,limit", [(1, 32, 64, 0.7), (17, 96, 192, 1.1), (40, 224, 128, 2.5), (140, 1088, 256, 0.9)])
def test_clamped_gated_unit(route, m, ff, k, limit):
    """Gate above the limit is cut, below it is not; up is cut on both sides; constants other than the design's."""
    rng = np.random.default_rng(ff + m)
    alpha, shift = 1.3, 0.75
    at, a = bf16_cuda(rng.standard_normal((m, k)))
    if route == "f32":
        at = f32(a)
    _, g = bf16_cuda(2.0 * rng.standard_normal((ff, k)) / np.sqrt(k))
    _, u = bf16_cuda(2.0 * rng.standard_normal((ff, k)) / np.sqrt(k))
    bg, bu = rng.standard_normal(ff).astype(np.float32), rng.standard_normal(ff).astype(np.float32)
    gz, uz = a.astype(np.float64) @ g.T + bg, a.astype(np.float64) @ u.T + bu
    assert (gz > limit).any() and (gz < -limit).any() and (uz > limit).any() and (uz < -limit).any()
    gc, uc = np.minimum(gz, limit), np.clip(uz, -limit, limit)
    ref = gc / (1.0 + np.exp(-alpha * gc)) * (uc + shift)
    wt, _ = bf16_cuda(interleave(g, u))
    got = to_np(ops.linear_act(at, wt, f32(interleave(bg[:, None], bu[:, None])[:, 0]), ops.EPI_GLU_CLAMP, (alpha, limit, shift), small=route == "small"))
    assert np.abs(got - ref).max() <= (2e-5 if route == "f32" else 1e-2) * np.abs(ref).max()


@pytest.mark.parametrize("kind", ["small", "f32"])
@pytest.mark.parametrize("m,heads,n,k", [(1, 3, 64, 128), (5, 20, 192, 64), (40, 7, 576, 256), (100, 2, 64, 512)])
def test_one_matrix_per_head(kind, m, heads, n, k):
    rng = np.random.default_rng(m + heads)
    at, a = bf16_cuda(rng.standard_normal((m, heads, k)))
    wt, w = bf16_cuda(rng.standard_normal((heads, n, k)) / np.sqrt(k))
    ref = np.einsum("mhk,hnk->mhn", a.astype(np.float64), w.astype(np.float64))
    if kind == "f32":
        assert np.abs(to_np(ops.linear_act(f32(a), wt, batch=heads)) - ref).max() <= 1e-5 * np.abs(ref).max()
    else:
        assert row_rel(to_np(ops.linear_act(at, wt, None, ops.EPI_BF16, small=True, batch=heads)), ref) <= 6e-3


@pytest.mark.parametrize("n,ld,snapshots", [(5, 64, 1), (136, 192, 3), (1000, 1024, 6), (2048, 2048, 29), (9000, 9024, 2)])
def test_depth_average_and_norm(n, ld, snapshots):
    rng = np.random.default_rng(n)
    hist = np.zeros((snapshots, 9, ld))
    hist[:, :, :n] = rng.standard_normal((snapshots, 9, n)) * 3
    coef, gain = rng.standard_normal(snapshots), np.zeros(ld)
    gain[:n] = rng.standard_normal(n)
    eps = 0.3   # large: a norm that leaves it out, or puts it outside the root, fails
    idx = np.array([8, 0, 3, 3], np.int32)
    for rows in (None, idx):
        x, inv, y = ops.depth_mix(f32(hist), f32(coef), f32(gain), n, eps, None if rows is None else i32(rows))
        h = hist if rows is None else hist[:, rows]
        ref = R.depth_mix(h, coef)
        assert np.abs(to_np(x) - ref).max() <= 1e-5 * np.abs(ref).max()
        norm = R.rms_norm(ref[:, :n], gain[:n], eps)
        assert np.abs(to_np(y)[:, :n] - norm).max() <= 1e-5 * np.abs(norm).max() and not to_np(y)[:, n:].any()
        assert np.abs(to_np(inv) * np.sqrt(np.mean(ref[:, :n] ** 2, 1) + eps) - 1).max() <= 1e-5
    with pytest.raises(ops.InvalidOp):
        ops.depth_mix(f32(hist), f32(coef), f32(gain), n, eps, i32([9]))


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6, 8])
def test_input_convolution_carries_its_state(taps):
    """Ragged steps of sequences in slots, cut anywhere (single tokens, fewer than the state holds, runs across the
    eight-row register blocks), against the convolution of the whole sequence; a slot that is used again starts
    from zeros; a decode step through the fused launch."""
    rng = np.random.default_rng(taps)
    n, ld, eps, slots = 132, 192, 1e-3, 5
    gain = np.zeros(ld)
    gain[:n] = 1 + 0.3 * rng.standard_normal(n)
    w = np.zeros((2, taps, ld))
    w[:, :, :n] = rng.standard_normal((2, taps, n))
    state = torch.zeros((slots, 2, taps - 1, ld), dtype=torch.float32, device=DEV)
    state += 7.0  # leftovers of earlier users
    phase = np.zeros(slots, np.uint8)
    seqs = {}

    def step(parts, fused=False):
        xs, cu, sid = [], [0], []
        for slot, k, fresh in parts:
            new = np.zeros((k, ld))
            new[:, :n] = rng.standard_normal((k, n)) * 2
            seqs[slot] = new if fresh else np.concatenate([seqs[slot], new])
            xs.append(new); cu.append(cu[-1] + k); sid += [len(cu) - 2] * k
        x = f32(np.concatenate(xs))
        sl, fr, ph = i32([p[0] for p in parts]), u8([p[2] for p in parts]), u8(phase[[p[0] for p in parts]])
        if fused:
            x2, o1, o2 = ops.depth_mix_conv_decode(x[None].contiguous(), f32([1.0]), f32(gain), f32(w[0]), f32(w[1]), state, sl, fr, ph, n, eps)
            assert torch.equal(x2, x)
        else:
            _, inv, _ = ops.depth_mix(x[None].contiguous(), f32([1.0]), f32(gain), n, eps)
            o1, o2 = ops.norm_conv(x, inv, f32(gain), f32(w[0]), f32(w[1]), state, sl, fr, ph, i32(sid), i32(cu))
        for (slot, k, _), a, b in zip(parts, cu, cu[1:]):
            h = R.rms_norm(seqs[slot][:, :n], gain[:n], eps)
            for o, f in ((o1, w[0]), (o2, w[1])):
                ref = (h + R.causal_conv(h, f[:, :n].T))[-k:]
                assert np.abs(to_np(o)[a:b, :n] - ref).max() <= 2e-5 * max(1.0, np.abs(ref).max()), (slot, k)
                assert not to_np(o)[a:b, n:].any()
            phase[slot] ^= 1

    step([(0, 1, 1), (3, 2, 1), (1, 19, 1)])
    step([(3, 1, 0), (0, 1, 0), (4, 9, 1)])
    step([(0, 1, 0), (1, 1, 0), (3, 1, 0)], fused=True)
    step([(4, 2, 0), (1, 3, 0), (0, 17, 0), (3, 1, 0)])
    step([(4, 1, 0), (2, 1, 1)], fused=True)
    step([(1, 1, 1), (4, 1, 0), (2, 1, 0)], fused=True)     # slot 1 again
    step([(1, 2, 0), (2, 11, 0)])


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-5), (torch.bfloat16, 6e-3)])
@pytest.mark.parametrize("qn,qw,cn,cw", [(40, 64, 72, 128), (96, 128, 200, 256), (1536, 1536, 512, 512)])
def test_latent_norm_and_store(dtype, tol, qn, qw, cn, cw):
    rng = np.random.default_rng(qn)
    rows, blocks, eps = 21, 6, 0.2
    raw = np.zeros((rows, qw + cw))
    raw[:, :qn] = rng.standard_normal((rows, qn))
    raw[:, qw:qw + cn] = rng.standard_normal((rows, cn)) * 2
    gq, gc = np.zeros(qw), np.zeros(cw)
    gq[:qn], gc[:cn] = rng.standard_normal(qn), rng.standard_normal(cn)
    pool = torch.full((blocks, 16, cw), 3.0, dtype=dtype, device=DEV)
    slots = rng.permutation(blocks * 16)[:rows]
    cq = to_np(ops.latent_norm_store(f32(raw), f32(gq), f32(gc), pool, torch.from_numpy(slots.astype(np.int64)).to(DEV), qn, cn, eps))
    flat = to_np(pool).reshape(-1, cw)
    assert row_rel(cq[:, :qn], R.rms_norm(raw[:, :qn], gq[:qn], eps)) <= tol and not cq[:, qn:].any()
    assert row_rel(flat[slots, :cn], R.rms_norm(raw[:, qw:qw + cn], gc[:cn], eps)) <= tol and not flat[slots, cn:].any()
    rest = np.setdiff1d(np.arange(blocks * 16), slots)
    assert (flat[rest] == 3.0).all()
    acc = f32(raw)
    assert np.array_equal(to_np(ops.latent_norm_store(acc, f32(gq), f32(gc), pool, torch.from_numpy(slots.astype(np.int64)).to(DEV), qn, cn, eps, zero_raw=True)), cq)
    assert not to_np(acc).any()
    with pytest.raises(ops.InvalidOp):
        ops.latent_norm_store(f32(raw[:1]), f32(gq), f32(gc), pool, torch.tensor([blocks * 16], device=DEV), qn, cn, eps)


def paged(rng, lens, rank, dtype):
    """Random cached latents of several sequences scattered over a pool: (pool, tables, per-sequence rows)."""
    need = [-(-n // 16) for n in lens]
    blocks = sum(need) + 3
    perm = rng.permutation(blocks)
    tables = np.full((len(lens), max(need) + 1), -1, np.int32)
    pool = rng.standard_normal((blocks, 16, rank))
    if dtype == torch.bfloat16:
        pool = R.bf16(pool)
    rows, at = [], 0
    for i, n in enumerate(lens):
        tables[i, :need[i]] = perm[at:at + need[i]]
        at += need[i]
        rows.append(np.concatenate([pool[b] for b in tables[i, :need[i]]])[:n])
    return pool, tables, rows


def test_latent_gather_places_every_sequence():
    rng = np.random.default_rng(0)
    lens = [1, 16, 17, 130, 8, 63]
    pool, tables, rows = paged(rng, lens, 192, torch.bfloat16)
    out, start = ops.latent_gather(bf16_cuda(pool)[0], i32(tables), i32(lens), lens)
    out, start = to_np(out), start.cpu().numpy()
    seen = np.zeros(out.shape[0], bool)
    for r, s in zip(rows, start):
        assert s % 8 == 0 and np.array_equal(out[s:s + len(r)], r)
        seen[s:s + len(r)] = True
    assert not out[~seen].any()
    tables[1, 0] = pool.shape[0]
    with pytest.raises(ops.InvalidOp):
        ops.latent_gather(bf16_cuda(pool)[0], i32(tables), i32(lens), lens)


LENS = [1, 2, 15, 16, 17, 63, 64, 65, 255, 256, 257, 700]


def make_queries(rng, rows, heads, rank, far):
    """Random queries; in every sequence each head's query matches one cached row so well that its score stands
    out: the first, the last, or the row at place far % length."""
    q = rng.standard_normal((len(rows), heads, rank)) * 0.3
    for i, c in enumerate(rows):
        for h in range(heads):
            k = (0, len(c) - 1, far % len(c))[h % 3]
            q[i, h] = c[k] * 0.6
    return q


def latent_attend(q, c, scale):
    s = np.einsum("hr,kr->hk", q, c) * scale
    p = np.exp(s - s.max(1, keepdims=True))
    return (p / p.sum(1, keepdims=True)) @ c


@pytest.mark.parametrize("heads,rank", [(3, 64), (16, 128), (20, 192), (8, 320), (16, 512), (33, 512), (70, 256), (5, 576), (18, 1024)])
@pytest.mark.parametrize("chunk", [0, 64])
def test_latent_decode_at_page_tile_and_chunk_borders(heads, rank, chunk):
    rng = np.random.default_rng(heads + rank)
    pool, tables, rows = paged(rng, LENS, rank, torch.bfloat16)
    scale = 12.0 / rank
    qt, q = bf16_cuda(make_queries(rng, rows, heads, rank, 100))
    got = to_np(ops.latent_decode(qt, bf16_cuda(pool)[0], i32(tables), i32(LENS), LENS, scale, chunk))
    for i, c in enumerate(rows):
        assert row_rel(got[i], latent_attend(q[i].astype(np.float64), c, scale)) <= TOL, LENS[i]
    # soft scores: every key counts
    qt, q = bf16_cuda(rng.standard_normal((len(LENS), heads, rank)) * 0.5)
    got = to_np(ops.latent_decode(qt, bf16_cuda(pool)[0], i32(tables), i32(LENS), LENS, 1.0 / rank, chunk))
    for i, c in enumerate(rows):
        assert row_rel(got[i], latent_attend(q[i].astype(np.float64), c, 1.0 / rank)) <= TOL, LENS[i]


@pytest.mark.parametrize("heads,rank", [(1, 64), (7, 192), (4, 1024)])
def test_latent_attention_f32(heads, rank):
    rng = np.random.default_rng(rank)
    pool, tables, rows = paged(rng, LENS, rank, torch.float32)
    pool = pool.astype(np.float32)
    seq, pos = [], []
    for i, n in enumerate(LENS):
        for p in {0, n // 2, max(0, n - 2), n - 1}:
            seq.append(i); pos.append(p)
    rows = [r.astype(np.float32).astype(np.float64) for r in rows]
    vis = [rows[s][:p + 1] for s, p in zip(seq, pos)]
    q = make_queries(rng, vis, heads, rank, 100).astype(np.float32)
    got = to_np(ops.latent_attention_f32(f32(q), f32(pool), i32(tables), i32(seq), i32(pos), 12.0 / rank))
    for i, c in enumerate(vis):
        assert row_rel(got[i], latent_attend(q[i].astype(np.float64), c, 12.0 / rank)) <= 2e-5


@pytest.mark.parametrize("D,heads,kv_heads", [(64, 5, 5), (64, 4, 2), (128, 3, 3), (256, 2, 2)])
def test_attention_over_contiguous_keys(D, heads, kv_heads):
    """Prefill chunks over prefixes of unequal length: first keys, far keys and keys at tile borders stand out; the
    last query of a chunk must see the whole sequence, the first nothing beyond itself."""
    rng = np.random.default_rng(D + heads)
    kv, new = [2, 130, 257, 600, 16, 128], [2, 130, 3, 140, 2, 127]
    starts, at = [], 0
    for n in kv:
        starts.append(at)
        at += (n + 7) // 8 * 8
    tp = (at + 15) // 16 * 16
    kt, k = bf16_cuda(rng.standard_normal((tp, kv_heads * D)))
    vt, v = bf16_cuda(rng.standard_normal((kv_heads * D, tp)))
    cu = np.concatenate([[0], np.cumsum(new)])
    q = rng.standard_normal((cu[-1], heads * D)) * 0.3
    scale = 9.0 / D
    for s in range(len(kv)):
        for i in range(new[s]):
            vis = kv[s] - new[s] + i + 1
            for h in range(heads):
                key = (0, vis - 1, max(0, vis - 129))[(h + i) % 3]
                kvh = h // (heads // kv_heads)
                q[cu[s] + i, h * D:(h + 1) * D] = k[starts[s] + key, kvh * D:(kvh + 1) * D] * 0.6
    qt, q = bf16_cuda(q)
    got = to_np(ops.attention_kv(qt, kt, vt, i32(cu), i32(kv), i32(starts), heads, kv_heads, D, scale, max(new)))
    for s in range(len(kv)):
        for h in range(heads):
            kvh = h // (heads // kv_heads)
            K = k[starts[s]:starts[s] + kv[s], kvh * D:(kvh + 1) * D].astype(np.float64)
            V = v[kvh * D:(kvh + 1) * D, starts[s]:starts[s] + kv[s]].T.astype(np.float64)
            full = np.zeros((kv[s], kv[s]))
            full[kv[s] - new[s]:] = q[cu[s]:cu[s + 1], h * D:(h + 1) * D].astype(np.float64) @ K.T * scale
            ref = (R.causal_softmax(full) @ V)[kv[s] - new[s]:]
            assert row_rel(got[cu[s]:cu[s + 1], h * D:(h + 1) * D], ref) <= TOL, (s, h)
