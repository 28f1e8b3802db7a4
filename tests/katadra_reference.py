"""A plain, slow statement of the Katadra decoder stack in float64 numpy, one function per mechanism, and seeded
random weights for it. It shares no code with the library: the GPU tests compare the executor and each of its
kernels with these functions.

Notation: one row per token; a matrix W of shape [out, in] is applied as W x. A layer's tensors are dicts keyed
by the name that follows its prefix."""
import numpy as np

from latent_reference import bf16, bf16_bits, write_checkpoint  # noqa: F401  (number format, model folder)


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def unit_rms(x, eps):
    """x divided by its root mean square over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def layer_norm(x, w, b, eps):
    m = np.mean(x, axis=-1, keepdims=True)
    return (x - m) / np.sqrt(np.mean((x - m) ** 2, axis=-1, keepdims=True) + eps) * w + b


# ---- attention with a soft cap and a learned bias of the distance ----------------------------------

def distance_bucket(n, buckets, far):
    """The row of the bias table for a distance n: one per distance below buckets // 2, then logarithmic up to `far`."""
    half = buckets // 2
    if n < half:
        return n
    return min(buckets - 1, half + int(np.floor(np.log(n / half) / np.log(far / half) * (buckets - half))))


def query_temperature(p, coef, every):
    return 1.0 + coef * np.log(np.floor((p + 1) / every) + 1.0)


def attention_scores(q, k, scale, cap, bias):
    """q, k [T, dim] of one head, bias [T] by distance; row i keeps columns 0..i (the rest is -inf)."""
    T = q.shape[0]
    s = cap * np.tanh(q @ k.T * scale / cap)
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return np.where(j <= i, s + bias[np.maximum(i - j, 0)], -np.inf)


def softmax(s):
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def bias_attention(h, w, m, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = unit_rms((h @ w["q"].T).reshape(T, H, m["dim"]), eps)
    k = unit_rms((h @ w["k"].T).reshape(T, G, m["dim"]), eps)
    v = (h @ w["v"].T).reshape(T, G, m["vdim"])
    q = q * np.array([query_temperature(p, m["q_temp"]["coef"], m["q_temp"]["every"]) for p in range(T)])[:, None, None]
    rows = [distance_bucket(n, w["rel"].shape[0], m["bias_max"]) for n in range(T)]
    o = np.zeros((T, H, m["vdim"]))
    for a in range(H):
        g = a // (H // G)
        o[:, a] = softmax(attention_scores(q[:, a], k[:, g], m["scale"], m["softcap"], w["rel"][rows, a])) @ v[:, g]
    return (o.reshape(T, -1) * sigmoid(h @ w["g"].T)) @ w["o"].T


# ---- time mixing -----------------------------------------------------------------------------------

def previous_rows(h):
    return np.concatenate([np.zeros_like(h[:1]), h[:-1]])


def time_mix_decay(x, w1, w2, w0):
    return np.exp(-np.exp(np.tanh(x @ w1.T) @ w2.T + w0))


def time_mix_recurrence(r, k, v, w, u, state=None):
    """r, k, w [T, D], v [T, V], u [D] of one head -> outputs [T, V] and the final state [D, V]."""
    S = np.zeros((r.shape[1], v.shape[1])) if state is None else state.copy()
    o = np.zeros((r.shape[0], v.shape[1]))
    for t in range(r.shape[0]):
        kv = np.outer(k[t], v[t])
        o[t] = (S + u[:, None] * kv).T @ r[t]
        S = w[t][:, None] * S + kv
    return o, S


def time_mix(h, w, m, eps):
    T, H, D = h.shape[0], m["heads"], m["dim"]
    d = previous_rows(h) - h
    mix = {s: h + d * w["mu." + s] for s in "rkvgw"}
    r, k, v = ((mix[s] @ w[s].T).reshape(T, H, D) for s in "rkv")
    decay = time_mix_decay(mix["w"], w["w1"], w["w2"], w["w0"]).reshape(T, H, D)
    o = np.stack([time_mix_recurrence(r[:, a], k[:, a], v[:, a], decay[:, a], w["u"][a])[0] for a in range(H)], axis=1)
    return (unit_rms(o, eps).reshape(T, -1) * w["norm"] * silu(mix["g"] @ w["g"].T)) @ w["o"].T


def parallel_mixer(h, w, m, eps):
    side = lambda s: {k[len(s) + 1:]: v for k, v in w.items() if k.startswith(s + ".")}
    return m["left_scale"] * bias_attention(h, side("left"), m["left"], eps) + m["right_scale"] * time_mix(h, side("right"), m["right"], eps)


# ---- state-space mixer -----------------------------------------------------------------------------

def causal_conv(x, w, b):
    """Depthwise over the rows of x [T, C] with w [C, taps]; rows before the first are zero."""
    T, taps = x.shape[0], w.shape[1]
    out = np.tile(b, (T, 1)).astype(np.float64)
    for t in range(T):
        for j in range(taps):
            if t - taps + 1 + j >= 0:
                out[t] += w[:, j] * x[t - taps + 1 + j]
    return out


def ssd_recurrence(x, B, C, dt, log_a, D, state=None):
    """x [T, V], B, C [T, N], dt [T] of one head, decay exp(-exp(log_a) dt) -> outputs [T, V], final state [N, V]."""
    S = np.zeros((B.shape[1], x.shape[1])) if state is None else state.copy()
    y = np.zeros_like(x)
    for t in range(x.shape[0]):
        S = np.exp(-np.exp(log_a) * dt[t]) * S + dt[t] * np.outer(B[t], x[t])
        y[t] = S.T @ C[t] + D * x[t]
    return y, S


def grouped_unit_rms(y, groups, eps):
    return unit_rms(y.reshape(y.shape[0], groups, -1), eps).reshape(y.shape)


def ssd_mixer(h, w, m, eps):
    T, H, V, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * V
    p = h @ w["in"].T
    z, xbc, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w["conv"], w["conv.b"]))
    x, B, C = xbc[:, :inner].reshape(T, H, V), xbc[:, inner:inner + G * N].reshape(T, G, N), xbc[:, inner + G * N:].reshape(T, G, N)
    dt = softplus(dt + w["dt_bias"])
    y = np.stack([ssd_recurrence(x[:, a], B[:, a // (H // G)], C[:, a // (H // G)], dt[:, a], w["A_log"][a], w["D"][a])[0] for a in range(H)], axis=1)
    y = grouped_unit_rms(y.reshape(T, -1) * silu(z), m["norm_groups"], eps)
    return (y * w["norm"]) @ w["o"].T


# ---- the stack -------------------------------------------------------------------------------------

def feed_forward(h, w):
    return np.maximum(h @ w["up"].T, 0.0) ** 2 @ w["down"].T


MIXERS = {"parallel": parallel_mixer, "mamba2": ssd_mixer}


def owner(cfg, i):
    """The layer whose tensors layer i uses."""
    while "weights_of" in cfg["layers"][i]:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of one whole sequence; layers_out (a list) receives the stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens, np.int64)]
    for i, lc in enumerate(cfg["layers"]):
        p = "l%d." % owner(cfg, i)
        part = lambda s: {k[len(p + s):]: v for k, v in w.items() if k.startswith(p + s)}
        y = MIXERS[lc["type"]](x, part("mix."), lc["mixer"], eps)
        x = x + layer_norm(y, w[p + "norm1"], w[p + "norm1.b"], eps)
        if lc["mlp"]:
            x = x + layer_norm(feed_forward(x, part("mlp.")), w[p + "norm2"], w[p + "norm2.b"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].T


def tensor_shapes(cfg, rel_rows=12, decay_rank=8):
    """Names and shapes; the rows of the bias tables and the rank of the decay are the tensors' own."""
    W = cfg["width"]
    s = {"embed": (cfg["vocab"], W), "final.norm": (W,), "final.norm.b": (W,), "head": (cfg["vocab"], W)}
    for i, lc in enumerate(cfg["layers"]):
        if "weights_of" in lc:
            continue
        p, m = "l%d." % i, lc["mixer"]
        s[p + "norm1"], s[p + "norm1.b"] = (W,), (W,)
        if lc["type"] == "mamba2":
            inner, gn = m["heads"] * m["vdim"], m["groups"] * m["state"]
            s[p + "mix.in"] = (2 * inner + 2 * gn + m["heads"], W)
            s[p + "mix.conv"], s[p + "mix.conv.b"] = (inner + 2 * gn, m["conv"]), (inner + 2 * gn,)
            for n in ("dt_bias", "A_log", "D"):
                s[p + "mix." + n] = (m["heads"],)
            s[p + "mix.norm"], s[p + "mix.o"] = (inner,), (W, inner)
        else:
            a, b = m["left"], m["right"]
            HV, HD = a["heads"] * a["vdim"], b["heads"] * b["dim"]
            q = p + "mix.left."
            s[q + "q"], s[q + "k"], s[q + "v"] = (a["heads"] * a["dim"], W), (a["kv_heads"] * a["dim"], W), (a["kv_heads"] * a["vdim"], W)
            s[q + "rel"], s[q + "g"], s[q + "o"] = (rel_rows, a["heads"]), (HV, W), (W, HV)
            q = p + "mix.right."
            for n in "rkvgw":
                s[q + "mu." + n] = (W,)
            for n in "rkvg":
                s[q + n] = (HD, W)
            s[q + "w1"], s[q + "w2"], s[q + "w0"] = (decay_rank, W), (HD, decay_rank), (HD,)
            s[q + "u"], s[q + "norm"], s[q + "o"] = (b["heads"], b["dim"]), (HD,), (W, HD)
        if lc["mlp"]:
            s[p + "norm2"], s[p + "norm2.b"] = (W,), (W,)
            s[p + "mlp.up"], s[p + "mlp.down"] = (lc["mlp"]["ff"], W), (W, lc["mlp"]["ff"])
    return s


def random_weights(cfg, seed, **sizes):
    """Seeded weights, every value representable in bfloat16: matrices of unit gain, gains and biases away from their
    neutral values, decays from nearly none to nearly total, so that a mechanism left out shows."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg, **sizes).items():
        z = rng.standard_normal(shape)
        leaf = name.split(".", 1)[1] if name[0] == "l" and name[1].isdigit() else name
        if leaf.endswith("norm.b") or leaf in ("norm1.b", "norm2.b"):
            v = 0.2 * z
        elif leaf.endswith("norm") or leaf in ("norm1", "norm2"):
            v = 1.0 + 0.3 * z
        elif ".mu." in leaf:
            v = 0.5 + 0.4 * z
        elif leaf.endswith(".rel"):
            v = 1.2 * z
        elif leaf.endswith(".u") or leaf.endswith("mix.D"):
            v = 0.7 * z
        elif leaf.endswith(".w0"):
            v = rng.uniform(-6.0, 1.0, shape)
        elif leaf.endswith("A_log"):
            v = rng.uniform(-2.0, 1.0, shape)
        elif leaf.endswith("dt_bias"):
            v = rng.uniform(-4.0, 0.5, shape)
        elif leaf.endswith("conv"):
            v = z / np.sqrt(shape[1])
        elif leaf.endswith("conv.b"):
            v = 0.2 * z
        elif name == "embed":
            v = z
        else:
            v = z / np.sqrt(shape[1])
        out[name] = bf16(v)
    return out
