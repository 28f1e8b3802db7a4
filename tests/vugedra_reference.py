"""A plain, slow statement of the Vugedra decoder stack in float64 numpy, one function per mechanism, and seeded
random weights for it. It shares no code with the library: the GPU tests compare the executor and each of its
kernels with these functions.

Notation: one row per token; a matrix W of shape [out, in] is applied as W x. A layer's tensors are dicts keyed
by the name that follows its prefix."""
import math

import numpy as np

from latent_reference import bf16, bf16_bits, write_checkpoint  # noqa: F401  (number format, model folder)


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def tanh_norm(x, alpha, w, b):
    """The norm of the stack: no statistics of the row."""
    return np.tanh(alpha * x) * w + b


# ---- rotary positions ------------------------------------------------------------------------------

def rotary_frequencies(rot):
    """Frequencies of the pairs of one head, and the factor on cosine and sine (YaRN interpolation: slow pairs are
    stretched by `factor`, fast ones kept, with a linear ramp between the pairs that turn `fast` and `slow` times
    over the original context)."""
    n, base = rot["dims"], rot["base"]
    f = base ** (-2.0 * np.arange(n // 2) / n)
    y = rot.get("scaling")
    if not y:
        return f, 1.0
    at = lambda turns: n * math.log(y["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(at(y["fast"])), 0), min(math.ceil(at(y["slow"])), n - 1)
    ramp = np.clip((np.arange(n // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / y["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(y["factor"]) + 1.0


def rotate(x, positions, rot):
    """x [T, heads, d]: neighbouring channels (2 i, 2 i + 1) of the first rot.dims are turned by position * f_i."""
    f, amp = rotary_frequencies(rot)
    a = np.asarray(positions, np.float64)[:, None, None] * f
    c, s = amp * np.cos(a), amp * np.sin(a)
    out = x.copy()
    n = rot["dims"]
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    out[..., 0:n:2], out[..., 1:n:2] = u * c - v * s, v * c + u * s
    return out


# ---- windowed attention ----------------------------------------------------------------------------

def window_mask(T, size, keep_first):
    """[T, T]: row i sees column j."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def softmax_plus_one(s):
    """Weights over the last axis with a further score of 0 in the denominator; -inf is not seen."""
    m = np.maximum(s.max(axis=-1, keepdims=True), 0.0)
    e = np.exp(s - m)
    return e / (np.exp(-m) + e.sum(axis=-1, keepdims=True))


def softmax(s):
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def window_attention_heads(q, k, v, scale, mask):
    """q [T, H, d], k [T, G, d], v [T, G, e], mask [T, T] -> [T, H, e]."""
    H, G = q.shape[1], k.shape[1]
    o = np.zeros((q.shape[0], H, v.shape[2]))
    for a in range(H):
        g = a // (H // G)
        o[:, a] = softmax_plus_one(np.where(mask, q[:, a] @ k[:, g].T * scale, -np.inf)) @ v[:, g]
    return o


def attention_qkv(h, w, m, eps):
    """Normed over the whole projection, split into heads and rotated: what the scores are made of."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = rms_norm(h @ w["q"].T + w["q.b"], w["q.norm"], eps).reshape(T, H, m["dim"])
    k = rms_norm(h @ w["k"].T + w["k.b"], w["k.norm"], eps).reshape(T, G, m["dim"])
    v = (h @ w["v"].T + w["v.b"]).reshape(T, G, m["vdim"])
    return rotate(q, np.arange(T), m["rot"]), rotate(k, np.arange(T), m["rot"]), v


def attention(h, w, m, eps):
    T = h.shape[0]
    q, k, v = attention_qkv(h, w, m, eps)
    o = window_attention_heads(q, k, v, m["scale"], window_mask(T, m["mask"]["size"], m["mask"]["keep_first"]))
    return (o * sigmoid(h @ w["g"].T)[:, :, None]).reshape(T, -1) @ w["o"].T


# ---- latent attention ------------------------------------------------------------------------------

def latent_cache_rows(h, w, m, eps):
    """What is kept of a token: its normed latent and the rotated key part that all heads share."""
    R = m["kv_rank"]
    raw = h @ w["dkv"].T
    return rms_norm(raw[:, :R], w["dkv.norm"], eps), rotate(raw[:, None, R:], np.arange(h.shape[0]), m["rot"])[:, 0]


def latent_queries(h, w, m, eps):
    """Unrotated and rotated part per head."""
    T, H, d = h.shape[0], m["heads"], m["dim"]
    q = (rms_norm(h @ w["dq"].T, w["dq.norm"], eps) @ w["uq"].T).reshape(T, H, d + m["rot_dim"])
    return q[..., :d], rotate(q[..., d:], np.arange(T), m["rot"])


def latent_attention(h, w, m, eps):
    T, H = h.shape[0], m["heads"]
    c, kr = latent_cache_rows(h, w, m, eps)
    qu, qr = latent_queries(h, w, m, eps)
    k, v = (c @ w["uk"].T).reshape(T, H, m["dim"]), (c @ w["uv"].T).reshape(T, H, m["vdim"])
    seen = np.tri(T, dtype=bool)
    o = np.stack([softmax(np.where(seen, (qu[:, a] @ k[:, a].T + qr[:, a] @ kr.T) * m["scale"], -np.inf)) @ v[:, a] for a in range(H)], axis=1)
    return (o * sigmoid(h @ w["g"].T)[:, :, None]).reshape(T, -1) @ w["o"].T


# ---- gated linear attention ------------------------------------------------------------------------

def log_decay(z, tau):
    return -np.logaddexp(0.0, -z) / tau


def gla_recurrence(q, k, v, alpha, state=None):
    """q, k, alpha [T, D], v [T, V] of one head -> outputs [T, V] and the final state [D, V]."""
    S = np.zeros((q.shape[1], v.shape[1])) if state is None else state.copy()
    o = np.zeros_like(v)
    for t in range(q.shape[0]):
        S = alpha[t][:, None] * S + np.outer(k[t], v[t])
        o[t] = S.T @ q[t]
    return o, S


def gla(h, w, m, eps):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w["q"].T).reshape(T, H, D) * D ** -0.5, (h @ w["k"].T).reshape(T, H, D), (h @ w["v"].T).reshape(T, H, V)
    alpha = np.exp(log_decay((h @ w["a1"].T) @ w["a2"].T + w["a2.b"], m["tau"])).reshape(T, H, D)
    o = np.stack([gla_recurrence(q[:, a], k[:, a], v[:, a], alpha[:, a])[0] for a in range(H)], axis=1)
    return (rms_norm(o, w["norm"], eps).reshape(T, -1) * silu(h @ w["g"].T)) @ w["o"].T


# ---- feed-forward ----------------------------------------------------------------------------------

def gated_unit(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def route(z, correction, top):
    """Router logits [T, n] -> the chosen experts [T, top] and their weights: chosen by softmax score plus correction,
    weighted by the scores alone."""
    s = softmax(z)
    chosen = np.argsort(-(s + correction), axis=-1, kind="stable")[:, :top]
    picked = np.take_along_axis(s, chosen, axis=-1)
    return chosen, picked / (picked.sum(axis=-1, keepdims=True) + 1e-20)


def mixture(h, w, c):
    part = lambda p: {n: w["%s.%s" % (p, n)] for n in ("gate", "up", "down")}
    r = c["router"]
    chosen, weight = route(h @ w["router"].T, w["correction"], r["top"])
    out = np.zeros_like(h)
    for e in range(r["experts"] + r.get("identity", 0)):
        t, slot = np.nonzero(chosen == e)
        if t.size:
            out[t] += weight[t, slot][:, None] * (gated_unit(h[t], part("e%d" % e)) if e < r["experts"] else h[t])
    return out + gated_unit(h, part("shared")) if c.get("shared") else out


def feed_forward(h, w, c):
    return gated_unit(h, w) if c["kind"] == "dense" else mixture(h, w, c)


# ---- the stack -------------------------------------------------------------------------------------

MIXERS = {"attention": attention, "gla": gla, "latent_attention": latent_attention}


def owner(cfg, i):
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of one whole sequence; layers_out (a list) receives the stream after every layer."""
    eps = cfg["norm"]["eps"]
    norm = lambda name, x: tanh_norm(x, w[name + ".alpha"], w[name], w[name + ".b"])
    x = w["embed"][np.asarray(tokens, np.int64)]
    for i, lc in enumerate(cfg["layers"]):
        p = "l%d." % owner(cfg, i)
        part = lambda s: {k[len(p + s):]: v for k, v in w.items() if k.startswith(p + s)}
        x = x + norm(p + "norm1b", MIXERS[lc["type"]](norm(p + "norm1", x), part("mix."), lc["mixer"], eps))
        if lc["mlp"]:
            x = x + norm(p + "norm2b", feed_forward(norm(p + "norm2", x), part("mlp."), lc["mlp"]))
        if layers_out is not None:
            layers_out.append(x)
    return norm("final.norm", x) @ w["head"].T


def tensor_shapes(cfg, decay_rank=8):
    """Names and shapes; the rank of the decay is the tensors' own."""
    W = cfg["width"]
    s = {"embed": (cfg["vocab"], W), "head": (cfg["vocab"], W)}

    def norm(name):
        s[name], s[name + ".b"], s[name + ".alpha"] = (W,), (W,), ()

    def unit(p, ff):
        s[p + "gate"], s[p + "up"], s[p + "down"] = (ff, W), (ff, W), (W, ff)

    norm("final.norm")
    for i, lc in enumerate(cfg["layers"]):
        if lc.get("weights_of") is not None:
            continue
        p, m, f = "l%d." % i, lc["mixer"], lc["mlp"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if f else ()):
            norm(p + n)
        q, H = p + "mix.", m["heads"]
        if lc["type"] == "attention":
            for n, rows in (("q", H * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
                s[q + n], s[q + n + ".b"] = (rows, W), (rows,)
                if n != "v":
                    s[q + n + ".norm"] = (rows,)
            s[q + "g"], s[q + "o"] = (H, W), (W, H * m["vdim"])
        elif lc["type"] == "gla":
            s[q + "q"], s[q + "k"], s[q + "v"], s[q + "g"] = (H * m["dim"], W), (H * m["dim"], W), (H * m["vdim"], W), (H * m["vdim"], W)
            s[q + "a1"], s[q + "a2"], s[q + "a2.b"] = (decay_rank, W), (H * m["dim"], decay_rank), (H * m["dim"],)
            s[q + "norm"], s[q + "o"] = (m["vdim"],), (W, H * m["vdim"])
        else:
            Q, R, r = m["q_rank"], m["kv_rank"], m["rot_dim"]
            s[q + "dq"], s[q + "dq.norm"], s[q + "uq"] = (Q, W), (Q,), (H * (m["dim"] + r), Q)
            s[q + "dkv"], s[q + "dkv.norm"] = (R + r, W), (R,)
            s[q + "uk"], s[q + "uv"] = (H * m["dim"], R), (H * m["vdim"], R)
            s[q + "g"], s[q + "o"] = (H, W), (W, H * m["vdim"])
        if not f:
            continue
        if f["kind"] == "dense":
            unit(p + "mlp.", f["ff"])
            continue
        n = f["router"]["experts"] + f["router"].get("identity", 0)
        for e in range(f["router"]["experts"]):
            unit(p + "mlp.e%d." % e, f["expert"]["ff"])
        s[p + "mlp.router"], s[p + "mlp.correction"] = (n, W), (n,)
        if f.get("shared"):
            unit(p + "mlp.shared.", f["shared"]["ff"])
    return s


def random_weights(cfg, seed, **sizes):
    """Seeded weights, every value representable in bfloat16: matrices of unit gain, gains and biases away from their
    neutral values, decays from nearly none to strong, so that a mechanism left out shows."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg, **sizes).items():
        z = rng.standard_normal(shape)
        if name.endswith(".alpha"):
            v = rng.uniform(0.5, 1.2)
        elif name.endswith(".a2.b"):
            v = rng.uniform(-4.0, 4.0, shape)
        elif name.endswith(".b"):
            v = 0.2 * z
        elif name.endswith("correction"):
            v = 0.15 * z
        elif len(shape) == 1:
            v = 1.0 + 0.3 * z
        elif name == "embed":
            v = z
        else:
            v = z / np.sqrt(shape[1])
        out[name] = bf16(np.asarray(v, np.float64)).reshape(shape)
    return out
