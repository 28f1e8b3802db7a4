"""A plain, slow statement of the latent-attention decoder stack in float64 numpy, one function per
mechanism, and seeded random weights for it. It shares no code with the library: the GPU tests compare
the executor and each of its kernels with these functions.

Notation: H = width, one row per token; a matrix W of shape [out, in] is applied as W x."""
import numpy as np


def bf16(x):
    """Rounds to bfloat16 (nearest even), returned as float64."""
    a = np.ascontiguousarray(x, dtype=np.float32)
    u = a.view(np.uint32).astype(np.uint64)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000
    return u.astype(np.uint32).view(np.float32).reshape(a.shape).astype(np.float64)


def bf16_bits(x):
    """The bfloat16 encoding (uint16) of values that are bfloat16 already."""
    return (np.ascontiguousarray(x, dtype=np.float32).view(np.uint32) >> 16).astype(np.uint16)


def rms_norm(x, gain, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * gain


def causal_conv(h, w):
    """Depthwise causal convolution along the rows of h [T, H] with w [H, taps]; rows before the first are zero."""
    taps = w.shape[1]
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(taps):
            src = t - taps + 1 + j
            if src >= 0:
                out[t] += w[:, j] * h[src]
    return out


def depth_mix(history, coef):
    return sum(c * x for c, x in zip(coef, history))


def latent_kv(h, w_dkv, gain, eps):
    return rms_norm(h @ w_dkv.T, gain, eps)


def latent_query(h, w_dq, gain, w_uq, heads, eps):
    q = rms_norm(h @ w_dq.T, gain, eps) @ w_uq.T
    return q.reshape(h.shape[0], heads, -1)


def causal_softmax(scores):
    """scores [T, T]: row i keeps columns 0..i."""
    out = np.zeros_like(scores)
    for i in range(scores.shape[0]):
        s = scores[i, :i + 1]
        e = np.exp(s - s.max())
        out[i, :i + 1] = e / e.sum()
    return out


def latent_attention(h, w, mixer, eps):
    """w: the layer's tensors by the names dq, dq.norm, uq, dkv, dkv.norm, uk, uv, o."""
    H = mixer["heads"]
    c = latent_kv(h, w["dkv"], w["dkv.norm"], eps)
    q = latent_query(h, w["dq"], w["dq.norm"], w["uq"], H, eps)
    k = (c @ w["uk"].T).reshape(-1, H, mixer["dim"])
    v = (c @ w["uv"].T).reshape(-1, H, mixer["vdim"])
    o = np.zeros((h.shape[0], H, mixer["vdim"]))
    for a in range(H):
        o[:, a] = causal_softmax(q[:, a] @ k[:, a].T * mixer["scale"]) @ v[:, a]
    return o.reshape(h.shape[0], -1) @ w["o"].T


def clamped_glu(h, w, limit):
    g = np.minimum(h @ w["gate"].T + w["gate.b"], limit)
    u = np.clip(h @ w["up"].T + w["up.b"], -limit, limit)
    y = g / (1.0 + np.exp(-1.702 * g)) * (u + 1.0)
    return y @ w["down"].T + w["down.b"]


def softcap(z, cap):
    return cap * np.tanh(z / cap)


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of one whole sequence; layers_out (a list) receives the stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens, np.int64)]
    history = [x]
    for i, lc in enumerate(cfg["layers"]):
        p = "l%d." % i
        mix = {k[len(p) + 4:]: v for k, v in w.items() if k.startswith(p + "mix.")}
        h = rms_norm(x, 1.0 + w[p + "norm1"], eps)
        y = latent_attention(h + causal_conv(h, w[p + "canon1"]), mix, lc["mixer"], eps)
        if lc.get("mlp"):
            mlp = {k[len(p) + 4:]: v for k, v in w.items() if k.startswith(p + "mlp.")}
            y = y + clamped_glu(h + causal_conv(h, w[p + "canon2"]), mlp, lc["mlp"]["limit"])
        history.append(x + y)
        x = depth_mix(history, w[p + "dwa"])
        if layers_out is not None:
            layers_out.append(x)
    z = rms_norm(x, 1.0 + w["final.norm"], eps) @ w["head"].T
    return softcap(z, cfg["logit_softcap"])


def tensor_shapes(cfg):
    H, taps = cfg["width"], cfg["canon"]["taps"]
    s = {"embed": (cfg["vocab"], H), "final.norm": (H,), "head": (cfg["vocab"], H)}
    for i, lc in enumerate(cfg["layers"]):
        m, p = lc["mixer"], "l%d." % i
        s[p + "norm1"] = (H,)
        s[p + "mix.dq"], s[p + "mix.dq.norm"] = (m["q_rank"], H), (m["q_rank"],)
        s[p + "mix.uq"] = (m["heads"] * m["dim"], m["q_rank"])
        s[p + "mix.dkv"], s[p + "mix.dkv.norm"] = (m["kv_rank"], H), (m["kv_rank"],)
        s[p + "mix.uk"], s[p + "mix.uv"] = (m["heads"] * m["dim"], m["kv_rank"]), (m["heads"] * m["vdim"], m["kv_rank"])
        s[p + "mix.o"] = (H, m["heads"] * m["vdim"])
        s[p + "canon1"], s[p + "dwa"] = (H, taps), (i + 2,)
        if lc.get("mlp"):
            f = lc["mlp"]["ff"]
            s[p + "canon2"] = (H, taps)
            s[p + "mlp.gate"], s[p + "mlp.gate.b"], s[p + "mlp.up"], s[p + "mlp.up.b"] = (f, H), (f,), (f, H), (f,)
            s[p + "mlp.down"], s[p + "mlp.down.b"] = (H, f), (H,)
    return s


def random_weights(cfg, seed):
    """Seeded weights, every value representable in bfloat16: matrices of unit gain, norm gains and depth
    coefficients away from 1, so that a mechanism left out shows."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        z = rng.standard_normal(shape)
        leaf = name.split(".", 1)[1] if "." in name else name
        if leaf in ("norm1", "norm"):                   # offsets from 1
            v = 0.3 * z
        elif name.endswith((".dq.norm", ".dkv.norm")):  # plain gains
            v = 1.0 + 0.3 * z
        elif leaf == "dwa":
            v = 0.25 * z
            v[-1] += 1.0
        elif leaf.startswith("canon"):
            v = 0.4 * z
        elif name.endswith(".b"):
            v = 0.2 * z
        elif name == "embed":
            v = z
        else:
            gain = 1.5 if leaf in ("mix.uq", "mix.uk") else 1.0
            v = gain * z / np.sqrt(shape[1])
        out[name] = bf16(v)
    return out


def write_checkpoint(path, cfg, w):
    """A model folder: config.json and model.safetensors (bfloat16, tensors back to back)."""
    import json
    import os
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    header, blobs, at = {}, [], 0
    for name, v in w.items():
        b = bf16_bits(v).tobytes()
        header[name] = {"dtype": "BF16", "shape": list(v.shape), "data_offsets": [at, at + len(b)]}
        blobs.append(b)
        at += len(b)
    h = json.dumps(header).encode()
    h += b" " * (-len(h) % 8)
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(len(h).to_bytes(8, "little") + h + b"".join(blobs))
