"""A plain, slow statement of the Zetalorn decoder stack in float64 numpy, one function per mechanism, and seeded random
weights for it. It shares no code with the library: the GPU tests compare the executor and each of its kernels with these
functions.

Notation: one row per token; a matrix W of shape [out, in] is applied as W x. A layer's tensors are dicts keyed by the name
that follows its prefix."""
import numpy as np

from latent_reference import bf16, bf16_bits, write_checkpoint  # noqa: F401  (number format, model folder)


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def gated_residual(x, y, h, w, b):
    """The stream after a sublayer with input h and result y."""
    return x + y * sigmoid(h @ w.T + b)


# ---- rotary positions ------------------------------------------------------------------------------

def rotary_frequencies(rot):
    n = rot["dims"]
    f = rot["base"] ** (-2.0 * np.arange(n // 2) / n)
    return f / rot["scaling"]["factor"] if rot.get("scaling") else f


def rotate(x, positions, rot, halves):
    """x [T, heads, d]: the first rot.dims channels of every head turned in pairs (2 i, 2 i + 1), or (i, i + dims / 2)."""
    a = np.asarray(positions, np.float64)[:, None, None] * rotary_frequencies(rot)
    c, s = np.cos(a), np.sin(a)
    out, n = x.copy(), rot["dims"]
    first = np.arange(n // 2) if halves else np.arange(0, n, 2)
    second = first + (n // 2 if halves else 1)
    u, v = x[..., first], x[..., second]
    out[..., first], out[..., second] = u * c - v * s, v * c + u * s
    return out


# ---- attention -------------------------------------------------------------------------------------

def softmax(s):
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def chunk_mask(T, size):
    """[T, T]: row i sees column j, both in one chunk."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & (i // size == j // size)


def window_mask(T, size):
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & (i - j < size)


def pooled_mask(T, size, pool):
    """[T, blocks]: row i sees a block once its last token has left the window."""
    i, b = np.arange(T)[:, None], np.arange(T // pool)[None, :]
    return b * pool + pool - 1 <= i - size


def pooled(x, pool):
    """Means over the whole blocks of x [T, heads, d]."""
    n = x.shape[0] // pool
    return x[:n * pool].reshape(n, pool, *x.shape[1:]).mean(axis=1)


def attend(q, k, v, scale, mask):
    """q [T, H, d], k [K, G, d], v [K, G, e], mask [T, K] -> [T, H, e]."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    o = np.zeros((T, H, v.shape[2]))
    for a in range(H):
        g = a // (H // G)
        o[:, a] = softmax(np.where(mask, q[:, a] @ k[:, g].T * scale, -np.inf)) @ v[:, g]
    return o


def pooled_window_attention(q, k, v, scale, size, pool):
    """A window of tokens and one key and value per block that lies before it, under one softmax."""
    T = q.shape[0]
    keys, values = np.concatenate([pooled(k, pool), k]), np.concatenate([pooled(v, pool), v])
    return attend(q, keys, values, scale, np.concatenate([pooled_mask(T, size, pool), window_mask(T, size)], axis=1))


def difference_weight(w, diff):
    return float(np.exp(np.sum(w["lq1"] * w["lk1"])) - np.exp(np.sum(w["lq2"] * w["lk2"])) + diff)


def difference(a1, a2, lam, diff, eps):
    """Of the outputs [T, H, e] of the two maps."""
    return rms(a1 - lam * a2, eps) * (1.0 - diff)


def attention_qkv(h, w, m, eps):
    """q [T, H, 2, d], k [T, G, 2, d], v [T, G, e] of the two maps."""
    T, d = h.shape[0], m["dim"]

    def maps(n, heads):
        x = rms((h @ w[n].T).reshape(T, heads * 2, d), eps) * w[n + ".norm"]
        return rotate(x, np.arange(T), m["rot"], halves=False).reshape(T, heads, 2, d)

    return maps("q", m["heads"]), maps("k", m["kv_heads"]), (h @ w["v"].T).reshape(T, m["kv_heads"], m["vdim"])


def attention(h, w, m, eps):
    """Differential attention over chunks."""
    T = h.shape[0]
    q, k, v = attention_qkv(h, w, m, eps)
    mask = chunk_mask(T, m["mask"]["size"])
    a1, a2 = (attend(q[:, :, i], k[:, :, i], v, m["scale"], mask) for i in range(2))
    return difference(a1, a2, difference_weight(w, m["diff"]), m["diff"], eps).reshape(T, -1) @ w["o"].T


def left_qkv(h, w, m, eps):
    T = h.shape[0]
    part = lambda n, heads: rotate(rms((h @ w[n].T).reshape(T, heads, m["dim"]), eps) * w[n + ".norm"], np.arange(T), m["rot"], halves=True)
    return part("q", m["heads"]), part("k", m["kv_heads"]), (h @ w["v"].T).reshape(T, m["kv_heads"], m["vdim"])


def left(h, w, m, eps):
    q, k, v = left_qkv(h, w, m, eps)
    o = pooled_window_attention(q, k, v, m["scale"], m["mask"]["size"], m["mask"]["pool"])
    return o.reshape(h.shape[0], -1) @ w["o"].T


# ---- linear attention with a fixed decay -----------------------------------------------------------

def decay_recurrence(q, k, v, decay, state=None):
    """q, k [T, D], v [T, V] of one head -> outputs [T, V] and the final state [D, V]."""
    S = np.zeros((q.shape[1], v.shape[1])) if state is None else state.copy()
    o = np.zeros_like(v)
    for t in range(q.shape[0]):
        S = decay * S + np.outer(k[t], v[t])
        o[t] = S.T @ q[t]
    return o, S


def right(h, w, m, eps):
    T, H = h.shape[0], m["heads"]
    q, k, v = (silu(h @ w[n].T).reshape(T, H, -1) for n in "qkv")
    o = np.stack([decay_recurrence(q[:, a], k[:, a], v[:, a], m["decay"][a])[0] for a in range(H)], axis=1).reshape(T, -1)
    return (rms(o, eps) * w["norm"] * sigmoid(h @ w["g"].T)) @ w["o"].T


def parallel(h, w, m, eps):
    side = lambda s: {k[len(s) + 1:]: v for k, v in w.items() if k.startswith(s + ".")}
    a, b = left(h, side("left"), m["left"], eps), right(h, side("right"), m["right"], eps)
    return 0.5 * (rms(a, eps) * w["left.out"] + rms(b, eps) * w["right.out"])


# ---- feed-forward ----------------------------------------------------------------------------------

def clamped_unit(h, w, limit):
    g, u = np.minimum(h @ w["gate"].T, limit), np.clip(h @ w["up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w["down"].T


def route(z, top, count, keep):
    """Router logits [T, n] -> the chosen experts [T, top] and their weights."""
    s = sigmoid(z)
    T, n = s.shape
    by_group = np.sort(s.reshape(T, count, n // count), axis=-1)[..., ::-1]
    best = np.argsort(-by_group[..., :2].sum(axis=-1), axis=-1, kind="stable")[:, :keep]
    open_ = np.zeros((T, count), bool)
    np.put_along_axis(open_, best, True, axis=1)
    chosen = np.argsort(-np.where(np.repeat(open_, n // count, axis=1), s, -1.0), axis=-1, kind="stable")[:, :top]
    picked = np.take_along_axis(s, chosen, axis=-1)
    return chosen, picked / (picked.sum(axis=-1, keepdims=True) + 1e-20)


def mixture(h, w, c):
    r = c["router"]
    chosen, weight = route(h @ w["router"].T, r["top"], r["groups"]["count"], r["groups"]["keep"])
    out = np.zeros_like(h)
    for e in range(r["experts"]):
        t, slot = np.nonzero(chosen == e)
        if t.size:
            out[t] += weight[t, slot][:, None] * clamped_unit(h[t], {n: w["e%d.%s" % (e, n)] for n in ("gate", "up", "down")}, c["expert"]["limit"])
    return out


# ---- the stack -------------------------------------------------------------------------------------

MIXERS = {"attention": attention, "parallel": parallel}


def runs(cfg):
    """(layer, pass or None) in the order of execution; the pass is named at its first layer."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    body = [(i, t if i == a else None) for t in range(loop["times"]) for i in range(a, b)]
    return [(i, None) for i in range(a)] + body + [(i, None) for i in range(b, n)]


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of one whole sequence; layers_out (a list) receives the stream after every layer run."""
    eps = cfg["norm"]["eps"]
    embedded = x = w["embed"][np.asarray(tokens, np.int64)]
    for i, t in runs(cfg):
        if t is not None:
            x = (x + embedded if t > 0 else x) + w["loop.step"][t]
        lc, p = cfg["layers"][i], "l%d." % i
        part = lambda s: {k[len(p + s):]: v for k, v in w.items() if k.startswith(p + s)}
        h = rms(x, eps) * w[p + "norm1"]
        x = gated_residual(x, MIXERS[lc["type"]](h, part("mix."), lc["mixer"], eps), h, w[p + "rg1"], w[p + "rg1.b"])
        if lc["mlp"]:
            h = rms(x, eps) * w[p + "norm2"]
            x = gated_residual(x, mixture(h, part("mlp."), lc["mlp"]), h, w[p + "rg2"], w[p + "rg2.b"])
        if layers_out is not None:
            layers_out.append(x)
    return rms(x, eps) * w["final.norm"] @ w["head"].T * cfg["logit_scale"]


def tensor_shapes(cfg):
    W = cfg["width"]
    s = {"embed": (cfg["vocab"], W), "head": (cfg["vocab"], W), "final.norm": ()}
    if cfg.get("loop"):
        s["loop.step"] = (cfg["loop"]["times"], W)
    for i, lc in enumerate(cfg["layers"]):
        p, m, f = "l%d." % i, lc["mixer"], lc["mlp"]
        for n in "12" if f else "1":
            s[p + "norm" + n], s[p + "rg" + n], s[p + "rg" + n + ".b"] = (), (W, W), (W,)
        q = p + "mix."
        if lc["type"] == "attention":
            H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            s[q + "q"], s[q + "k"], s[q + "v"], s[q + "o"] = (H * 2 * d, W), (G * 2 * d, W), (G * e, W), (W, H * e)
            for n in ("q.norm", "k.norm", "lq1", "lk1", "lq2", "lk2"):
                s[q + n] = (d,)
        else:
            a, b = m["left"], m["right"]
            H, G, d, e = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            s[q + "left.q"], s[q + "left.k"], s[q + "left.v"], s[q + "left.o"] = (H * d, W), (G * d, W), (G * e, W), (W, H * e)
            s[q + "left.q.norm"], s[q + "left.k.norm"], s[q + "left.out"] = (d,), (d,), (W,)
            H, d, e = b["heads"], b["dim"], b["vdim"]
            for n, rows in (("q", H * d), ("k", H * d), ("v", H * e), ("g", H * e)):
                s[q + "right." + n] = (rows, W)
            s[q + "right.norm"], s[q + "right.o"], s[q + "right.out"] = (H * e,), (W, H * e), (W,)
        if f:
            for e in range(f["router"]["experts"]):
                for n, shape in (("gate", (f["expert"]["ff"], W)), ("up", (f["expert"]["ff"], W)), ("down", (W, f["expert"]["ff"]))):
                    s[p + "mlp.e%d.%s" % (e, n)] = shape
            s[p + "mlp.router"] = (f["router"]["experts"], W)
    return s


def random_weights(cfg, seed):
    """Seeded weights, every value representable in bfloat16: matrices of unit gain, gains and biases away from their
    neutral values, so that a mechanism left out shows."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        z = rng.standard_normal(shape)
        if shape == ():
            v = rng.uniform(0.6, 1.4)
        elif name.endswith(".b"):
            v = 0.5 * z
        elif name[-3:-1] in ("lq", "lk"):
            v = z * 0.7 / np.sqrt(np.sqrt(shape[0]))
        elif name == "loop.step":
            v = 0.7 * z
        elif len(shape) == 1:
            v = 1.0 + 0.3 * z
        elif name == "embed":
            v = z
        else:
            v = z / np.sqrt(shape[1])
        out[name] = bf16(np.asarray(v, np.float64)).reshape(shape)
    return out
