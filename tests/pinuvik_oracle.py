"""Plain Pinuvik decoder in numpy float64: one function per mechanism, whole sequences
from position 0, no cache, no padding, no batching.  Written from the equations; it
shares no code with the package.

    x <- x + N1b(mixer(shift(N1(x)))),   x <- x + N2b(ff(N2(x)))
"""
import json
import struct

import numpy as np


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def token_shift(h, mu, before=None):
    """h_t + (h_{t-1} - h_t) * mu; before = h of the token ahead of the first (zeros)."""
    first = np.zeros_like(h[:1]) if before is None else before[None]
    prev = np.concatenate([first, h[:-1]])
    return h + (prev - h) * mu


def rotate(x, positions, rot_dims, base):
    """x [T, heads, dim]; channels (2i, 2i + 1), i < rot_dims / 2, turn by
    p * base^(-2i / rot_dims)."""
    y = x.copy()
    for i in range(rot_dims // 2):
        ang = positions * float(base) ** (-2.0 * i / rot_dims)
        c, s = np.cos(ang)[:, None], np.sin(ang)[:, None]
        a, b = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        y[:, :, 2 * i] = a * c - b * s
        y[:, :, 2 * i + 1] = b * c + a * s
    return y


def visible(i, j, chunk):
    return j <= i and (chunk is None or i // chunk == j // chunk)


def attend(q, k, v, scale, chunk):
    """q [T, H, d], k / v [T, G, d]; query head h reads group h // (H / G)."""
    t, heads, _ = q.shape
    per = heads // k.shape[1]
    out = np.zeros((t, heads, v.shape[2]))
    for i in range(t):
        js = [j for j in range(i + 1) if visible(i, j, chunk)]
        for h in range(heads):
            s = np.array([q[i, h] @ k[j, h // per] for j in js]) * scale
            p = np.exp(s - s.max())
            out[i, h] = (p / p.sum()) @ v[js, h // per]
    return out


def chunked_attention(h, w, p, c, eps):
    t = h.shape[0]
    q = (h @ w[p + "q"].T).reshape(t, c["heads"], c["dim"])
    k = (h @ w[p + "k"].T).reshape(t, c["kv_heads"], c["dim"])
    v = k
    pos = np.arange(t, dtype=np.float64)
    qn = rms(rotate(q, pos, c["rot"]["dims"], c["rot"]["base"]), eps)
    kn = rms(rotate(k, pos, c["rot"]["dims"], c["rot"]["base"]), eps)
    o = attend(qn, kn, v, c["scale"], c["mask"]["size"])
    return o.reshape(t, -1) @ w[p + "o"].T


def delta_rule(r, k, v, decay, rate, state=None):
    """[T, heads, d] each; S <- diag(w) S - (a u)(u^T S) + k v^T, o = S^T r.
    Returns (o, last S [heads, d (key), d (value)])."""
    t, heads, d = k.shape
    s = np.zeros((heads, d, d)) if state is None else state.copy()
    o = np.zeros((t, heads, d))
    for i in range(t):
        for h in range(heads):
            u = k[i, h] / np.sqrt(np.sum(k[i, h] ** 2) + 1e-6)
            old = s[h]
            s[h] = decay[i, h][:, None] * old - np.outer(rate[i, h] * u, u @ old) \
                + np.outer(k[i, h], v[i, h])
            o[i, h] = s[h].T @ r[i, h]
    return o, s


def delta_decay(y1, w2, w0):
    return np.exp(-np.exp(-0.5) * sigmoid(np.tanh(y1) @ w2.T + w0))


def delta_mixer(h, w, p, c, eps):
    t, heads, d = h.shape[0], c["heads"], c["dim"]
    r, k, v = ((h @ w[p + n].T).reshape(t, heads, d) for n in "rkv")
    decay = delta_decay(h @ w[p + "w1"].T, w[p + "w2"], w[p + "w0"]).reshape(t, heads, d)
    rate = sigmoid(h @ w[p + "a"].T + w[p + "a.b"]).reshape(t, heads, d)
    o, _ = delta_rule(r, k, v, decay, rate)
    y = rms(o, eps).reshape(t, -1) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)
    return y @ w[p + "o"].T


def parallel_mixer(h, w, p, c, eps):
    a = rms(chunked_attention(h, w, p + "left.", c["left"], eps), eps) * w[p + "left.out"]
    b = rms(delta_mixer(h, w, p + "right.", c["right"], eps), eps) * w[p + "right.out"]
    return 0.5 * (a + b)


def feed_forward(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def layer_order(cfg):
    idx = list(range(len(cfg["layers"])))
    loop = cfg.get("loop")
    if not loop:
        return idx
    a, b = loop["start"], loop["stop"]
    out = idx[:a]
    for _ in range(loop["times"]):
        out += idx[a:b]
    return out + idx[b:]


def logits(cfg, w, tokens):
    """[T, vocab] for a whole sequence."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)]
    for i in layer_order(cfg):
        p, c = f"l{i}.", cfg["layers"][i]
        h = token_shift(rms(x, eps) * w[p + "norm1"], w[p + "shift"])
        x = x + rms(parallel_mixer(h, w, p + "mix.", c["mixer"], eps), eps) * w[p + "norm1b"]
        if c["mlp"] is not None:
            h = rms(x, eps) * w[p + "norm2"]
            x = x + rms(feed_forward(h, w, p + "mlp."), eps) * w[p + "norm2b"]
    return (rms(x, eps) * w["final.norm"]) @ w["head"].T


# ------------------------------------------------------------ small models for tests
def bf16(a):
    """Round to bf16 (nearest even), as float64."""
    u = np.asarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000
    return u.astype(np.uint32).view(np.float32).astype(np.float64)


def layer_config(heads=4, kv_heads=2, dim=32, chunk=24, rot=(16, 10000.0), scale=None,
                 delta=(3, 16), ff=72):
    return {"type": "parallel",
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim,
                               "mask": {"size": chunk}, "rot": {"dims": rot[0], "base": rot[1]},
                               "scale": dim ** -0.5 if scale is None else scale},
                      "right": {"heads": delta[0], "dim": delta[1]}},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def model_config(layers, width=96, vocab=203, eps=1e-5, loop=None):
    cfg = {"architecture": "Pinuvik", "layers": layers, "norm": {"eps": eps}, "vocab": vocab,
           "width": width}
    if loop is not None:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


# name: (configuration, rank of the decay's low-rank pair)
MODELS = {
    "plain": (model_config([layer_config(), layer_config(chunk=40, ff=None)], width=96), 10),
    "loop": (model_config([layer_config(heads=3, kv_heads=1, dim=20, rot=(8, 500.0), chunk=17,
                                            delta=(1, 40), ff=50, scale=0.6),
                             layer_config(heads=2, kv_heads=2, dim=56, rot=(56, 2e4), chunk=33,
                                            delta=(5, 8), ff=130),
                             layer_config(heads=4, kv_heads=4, dim=32, rot=(0, 1.0), chunk=17)],
                            width=72, vocab=131, eps=1e-3, loop=(1, 2, 3)), 5),
    "wide": (model_config([layer_config(heads=4, kv_heads=2, dim=128, rot=(64, 1e5), chunk=90,
                                            delta=(3, 64), ff=192, scale=0.2),
                             layer_config(heads=1, kv_heads=1, dim=136, rot=(136, 1e3), chunk=128,
                                            delta=(2, 72), ff=64)], width=320, vocab=500,
                            loop=(0, 2, 2)), 24),
}


def random_weights(cfg, seed, rank=10):
    """Weights of unit-scale activations; gains, shifts and biases away from 0 and 1."""
    rs = np.random.RandomState(seed)
    w, wd = {}, cfg["width"]

    def mat(name, n, k, gain=1.0):
        w[name] = bf16(rs.randn(n, k) * gain / np.sqrt(k))

    def vec(name, shape, lo, hi):
        w[name] = bf16(rs.uniform(lo, hi, size=shape))

    w["embed"] = bf16(rs.randn(cfg["vocab"], wd))
    mat("head", cfg["vocab"], wd)
    vec("final.norm", (), 0.7, 1.3)
    for i, c in enumerate(cfg["layers"]):
        p = f"l{i}."
        for n in ("norm1", "norm1b"):
            vec(p + n, (), 0.6, 1.4)
        vec(p + "shift", (wd,), 0.1, 0.8)
        left, right = c["mixer"]["left"], c["mixer"]["right"]
        m = p + "mix.left."
        mat(m + "q", left["heads"] * left["dim"], wd)
        mat(m + "k", left["kv_heads"] * left["dim"], wd)
        mat(m + "o", wd, left["heads"] * left["dim"])
        vec(m + "out", (wd,), 0.5, 1.5)
        m, hd = p + "mix.right.", right["heads"] * right["dim"]
        for n in "rkvga":
            mat(m + n, hd, wd)
        vec(m + "a.b", (hd,), -1.0, 1.0)
        mat(m + "w1", rank, wd)
        mat(m + "w2", hd, rank)
        vec(m + "w0", (hd,), -4.0, 1.0)
        vec(m + "norm", (hd,), 0.5, 1.5)
        mat(m + "o", wd, hd)
        vec(m + "out", (wd,), 0.5, 1.5)
        if c["mlp"] is not None:
            for n in ("norm2", "norm2b"):
                vec(p + n, (), 0.6, 1.4)
            mat(p + "mlp.gate", c["mlp"]["ff"], wd, 1.5)
            mat(p + "mlp.up", c["mlp"]["ff"], wd)
            mat(p + "mlp.down", wd, c["mlp"]["ff"])
    return w


def write_folder(folder, cfg, w):
    """config.json + model.safetensors (bf16) of a small model."""
    header, blobs, at = {}, [], 0
    for name, a in w.items():
        raw = (np.asarray(a, dtype=np.float32).view(np.uint32) >> 16).astype("<u2").tobytes()
        header[name] = {"dtype": "BF16", "shape": list(np.shape(a)),
                        "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    head = json.dumps(header).encode()
    (folder / "config.json").write_text(json.dumps(cfg))
    with open(folder / "model.safetensors", "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head + b"".join(blobs))
