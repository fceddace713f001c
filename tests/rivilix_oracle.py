"""Plain Rivilix decoder in numpy float64: one function per mechanism, whole sequences
from position 0, no cache, no padding, no batching.  Written from the equations; it
shares no code with the package.

    x <- x + mixer(LN1(x)) + ff(LN2(x))
"""
import json
import math
import struct

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def log_sigmoid(z):
    return -np.logaddexp(0.0, -z)


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def layer_norm(x, weight, bias, eps):
    mu = x.mean(-1, keepdims=True)
    var = np.mean((x - mu) ** 2, -1, keepdims=True)
    return (x - mu) / np.sqrt(var + eps) * weight + bias


def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """Row of the pair table for every token; the first token has no pair."""
    rows = [buckets]
    for a, b in zip(tokens[:-1], tokens[1:]):
        rows.append((int(a) * mul_prev + int(b) * mul_cur) % buckets)
    return np.array(rows, dtype=np.int64)


def embedding(tokens, w, bigram):
    x = w["embed"][tokens]
    if bigram:
        rows = bigram_rows(tokens, w["bigram"].shape[0] - 1, bigram["mul_prev"],
                           bigram["mul_cur"])
        x = x + w["bigram"][rows]
    return x


# ------------------------------------------------------------------- matrix memory
def mlstm_gates(zi, zf, cap):
    """Log input and log forget gate."""
    return cap * np.tanh(zi / cap), log_sigmoid(cap * np.tanh(zf / cap))


def mlstm_memory(q, k, v, i, f, state=None):
    """q, k [T, heads, dim], v [T, heads, vdim], i, f [T, heads]; o [T, heads, vdim] and
    the last (S, n, m)."""
    t, heads, dim = k.shape
    if state is None:
        state = np.zeros((heads, dim, v.shape[2])), np.zeros((heads, dim)), np.zeros(heads)
    s, n, m = (a.copy() for a in state)
    o = np.zeros(v.shape)
    for a in range(t):
        for h in range(heads):
            m_new = max(f[a, h] + m[h], i[a, h])
            keep, add = np.exp(f[a, h] + m[h] - m_new), np.exp(i[a, h] - m_new)
            s[h] = keep * s[h] + add * np.outer(k[a, h], v[a, h])
            n[h] = keep * n[h] + add * k[a, h]
            m[h] = m_new
            o[a, h] = (s[h].T @ q[a, h]) / (max(abs(n[h] @ q[a, h]), np.exp(-m_new)) + 1e-6)
    return o, (s, n, m)


def mlstm_mixer(h, w, p, c, eps):
    t, heads, dim, vdim = h.shape[0], c["heads"], c["dim"], c["vdim"]
    q = (h @ w[p + "q"].T).reshape(t, heads, dim) * dim ** -0.5
    k = (h @ w[p + "k"].T).reshape(t, heads, dim)
    v = (h @ w[p + "v"].T).reshape(t, heads, vdim)
    i, f = mlstm_gates(h @ w[p + "i"].T + w[p + "i.b"], h @ w[p + "f"].T + w[p + "f.b"],
                       c["gate_cap"])
    o, _ = mlstm_memory(q, k, v, i, f)
    y = rms(o, eps).reshape(t, -1) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)
    return y @ w[p + "o"].T


# ---------------------------------------------------------------- latent attention
def rotary_frequencies(dims, base, scaling=None):
    """(angle per position of every pair, factor on cos and sin)."""
    f = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return np.array(f), 1.0

    def turns(t):
        return dims * math.log(scaling["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo = max(math.floor(turns(scaling["fast"])), 0)
    hi = min(math.ceil(turns(scaling["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / scaling["factor"] * ramp + fi * (1.0 - ramp))
    return np.array(out), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x, positions, freqs, mscale):
    """x [T, ..., dims]: channels (2i, 2i + 1) turn by position * freqs[i]."""
    y = x.copy()
    for i, f in enumerate(freqs):
        shape = (-1,) + (1,) * (x.ndim - 2)
        c = (np.cos(positions * f) * mscale).reshape(shape)
        s = (np.sin(positions * f) * mscale).reshape(shape)
        a, b = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i] = a * c - b * s
        y[..., 2 * i + 1] = b * c + a * s
    return y


def causal_attention(q, k, v, scale):
    """q, k [T, H, d], v [T, H, e]."""
    t, heads, _ = q.shape
    out = np.zeros((t, heads, v.shape[2]))
    for h in range(heads):
        s = (q[:, h] @ k[:, h].T) * scale
        s[np.triu_indices(t, 1)] = -np.inf
        s = np.exp(s - s.max(-1, keepdims=True))
        out[:, h] = (s / s.sum(-1, keepdims=True)) @ v[:, h]
    return out


def latent_mixer(h, w, p, c, eps):
    t, heads, dim, rot, vdim = h.shape[0], c["heads"], c["dim"], c["rot_dim"], c["vdim"]
    q = (h @ w[p + "q"].T).reshape(t, heads, dim + rot)
    z = h @ w[p + "dkv"].T
    lat = rms(z[:, :c["kv_rank"]], eps) * w[p + "dkv.norm"]
    freqs, mscale = rotary_frequencies(rot, c["rot"]["base"], c["rot"].get("scaling"))
    pos = np.arange(t, dtype=np.float64)
    kr = rotate(z[:, c["kv_rank"]:], pos, freqs, mscale)
    qr = rotate(q[..., dim:], pos, freqs, mscale)
    k = (lat @ w[p + "uk"].T).reshape(t, heads, dim)
    v = (lat @ w[p + "uv"].T).reshape(t, heads, vdim)
    qq = np.concatenate([q[..., :dim], qr], -1)
    kk = np.concatenate([k, np.repeat(kr[:, None], heads, 1)], -1)
    return causal_attention(qq, kk, v, c["scale"]).reshape(t, -1) @ w[p + "o"].T


# -------------------------------------------------------------------- feed-forward
def gated(h, w, p, bias):
    g, u = h @ w[p + "gate"].T, h @ w[p + "up"].T
    if bias:
        g, u = g + w[p + "gate.b"], u + w[p + "up.b"]
    y = (silu(g) * u) @ w[p + "down"].T
    return y + w[p + "down.b"] if bias else y


def route(h, w, p, top):
    """(chosen experts [T, top], their weights)."""
    z = h @ w[p + "router"].T + w[p + "router.b"]
    chosen = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    zc = np.take_along_axis(z, chosen, -1)
    e = np.exp(zc - zc.max(-1, keepdims=True))
    return chosen, e / e.sum(-1, keepdims=True)


def mixture(h, w, p, c):
    chosen, weight = route(h, w, p, c["router"]["top"])
    y = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(chosen[t], weight[t]):
            y[t] += a * gated(h[t:t + 1], w, f"{p}e{e}.", False)[0]
    if c.get("shared"):
        y = y + gated(h, w, p + "shared.", False)
    return y


def feed_forward(h, w, p, c):
    if c.get("kind", "dense") == "moe":
        return mixture(h, w, p, c)
    return gated(h, w, p, True)


# ----------------------------------------------------------------------- the model
def layer_step(x, w, i, entry, eps):
    p = f"l{i}."
    mixer = {"mlstm": mlstm_mixer, "latent_attention": latent_mixer}[entry["type"]]
    y = mixer(layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps), w, p + "mix.",
              entry["mixer"], eps)
    if entry.get("mlp"):
        y = y + feed_forward(layer_norm(x, w[p + "norm2"], w[p + "norm2.b"], eps), w, p + "mlp.",
                             entry["mlp"])
    return x + y


def order(cfg):
    """[(layer, begins a pass of the loop)]"""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    body = [(i, i == a) for i in range(a, b)] * loop["times"]
    return [(i, False) for i in range(a)] + body + [(i, False) for i in range(b, n)]


def forward(tokens, w, cfg, layers=None):
    """Logits [T, vocab]; the residual after every layer run is appended to `layers`."""
    eps = cfg["norm"]["eps"]
    x = embedding(np.asarray(tokens), w, cfg.get("embedding", {}).get("bigram"))
    x0 = x
    for i, begins in order(cfg):
        if begins:
            x = np.concatenate([x, x0], -1) @ w["loop.in"].T
        x = layer_step(x, w, i, cfg["layers"][i], eps)
        if layers is not None:
            layers.append(x)
    z = layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].T
    cap = cfg.get("logit_softcap")
    return cap * np.tanh(z / cap) if cap else z


def bf16(a):
    """Nearest bfloat16 (ties to even), as float64."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & np.uint32(0xFFFF0000)
    return u.view(np.float32).astype(np.float64)


def read_safetensors(path):
    with open(path, "rb") as f:
        raw = f.read()
    n = struct.unpack("<Q", raw[:8])[0]
    out = {}
    for name, meta in json.loads(raw[8:8 + n]).items():
        if name == "__metadata__":
            continue
        a, b = meta["data_offsets"]
        data = raw[8 + n + a:8 + n + b]
        if meta["dtype"] == "BF16":
            v = (np.frombuffer(data, "<u2").astype(np.uint32) << 16).view(np.float32)
        else:
            v = np.frombuffer(data, {"F32": "<f4", "I32": "<i4"}[meta["dtype"]])
        out[name] = v.reshape(meta["shape"]).astype(np.float64)
    return out
