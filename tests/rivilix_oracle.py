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


def latent_attend(q, z, w, p, c, eps):
    """Heads' outputs [T, heads * vdim] from queries [T, heads, dim + rot] and latent rows
    [T, rank + rot]."""
    t, heads, dim, rot, vdim = q.shape[0], c["heads"], c["dim"], c["rot_dim"], c["vdim"]
    lat = rms(z[:, :c["kv_rank"]], eps) * w[p + "dkv.norm"]
    freqs, mscale = rotary_frequencies(rot, c["rot"]["base"], c["rot"].get("scaling"))
    pos = np.arange(t, dtype=np.float64)
    kr = rotate(z[:, c["kv_rank"]:], pos, freqs, mscale)
    qr = rotate(q[..., dim:], pos, freqs, mscale)
    k = (lat @ w[p + "uk"].T).reshape(t, heads, dim)
    v = (lat @ w[p + "uv"].T).reshape(t, heads, vdim)
    qq = np.concatenate([q[..., :dim], qr], -1)
    kk = np.concatenate([k, np.repeat(kr[:, None], heads, 1)], -1)
    return causal_attention(qq, kk, v, c["scale"]).reshape(t, -1)


def latent_mixer(h, w, p, c, eps):
    q = (h @ w[p + "q"].T).reshape(h.shape[0], c["heads"], -1)
    return latent_attend(q, h @ w[p + "dkv"].T, w, p, c, eps) @ w[p + "o"].T


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


# ------------------------------------------------------------ small models for tests
def memory_layer(heads=3, dim=20, vdim=28, cap=7.0, mlp=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim,
                                       "gate_cap": cap}, "mlp": mlp}


def latent_layer(heads=5, dim=24, rot=8, vdim=20, rank=40, scale=0.3, base=900.0, yarn=(4.0, 60, 8.0, 0.5),
                 mlp=None):
    r = {"base": base, "dims": rot}
    if yarn:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank,
                      "scale": scale, "rot": r}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def experts(n, top, ff, shared=None):
    c = {"kind": "moe", "router": {"experts": n, "top": top}, "expert": {"ff": ff}}
    if shared:
        c["shared"] = {"ff": shared}
    return c


def model_config(layers, width=104, vocab=201, eps=1e-4, loop=None, bigram=None, softcap=None):
    cfg = {"architecture": "Rivilix", "layers": layers, "norm": {"eps": eps}, "vocab": vocab,
           "width": width}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    if bigram:
        cfg["embedding"] = {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}
    if softcap:
        cfg["logit_softcap"] = softcap
    return cfg


MODELS = {
    "plain": model_config([memory_layer(mlp=dense(70)),
                           latent_layer(mlp=experts(7, 3, 36, shared=52)),
                           latent_layer(heads=2, rot=10, dim=15, vdim=33, rank=23, yarn=None,
                                        mlp=dense(90))],
                          bigram=(37, 11, 5), softcap=9.0),
    # the whole stack but its last layer repeats; a layer without feed-forward
    "loop": model_config([memory_layer(heads=2, dim=9, vdim=7, cap=3.0, mlp=experts(5, 1, 20)),
                          latent_layer(heads=1, dim=40, rot=40, vdim=8, rank=16, yarn=(1.0, 90, 4.0, 1.0)),
                          memory_layer(heads=1, dim=33, vdim=65, cap=20.0, mlp=dense(30))],
                         width=72, vocab=130, eps=1e-3, loop=(0, 2, 3), bigram=(64, 1, 3),
                         softcap=3.0),
    # heads beyond 128 channels, key sizes beyond 256, more heads than one tile of rows
    "wide": model_config([latent_layer(heads=3, dim=120, rot=40, vdim=136, rank=200, scale=0.12,
                                       mlp=experts(40, 5, 24, shared=100)),
                          memory_layer(heads=2, dim=264, vdim=72, mlp=None),
                          latent_layer(heads=19, dim=16, rot=2, vdim=16, rank=300, mlp=dense(64))],
                         width=200, vocab=300, loop=(1, 3, 2)),
    # a latent wider than the tensor-core kernels take
    "rank": model_config([latent_layer(heads=2, dim=32, rot=64, vdim=24, rank=620, scale=0.2,
                                       mlp=experts(2, 2, 30)),
                          memory_layer(heads=4, dim=4, vdim=3)], width=64, vocab=90,
                         bigram=(1, 7, 9)),
}


def random_weights(cfg, seed):
    """Weights of unit-scale activations: attention that picks few keys, memories that last,
    norms and biases away from 1 and 0."""
    rs = np.random.RandomState(seed)
    w, wd = {}, cfg["width"]

    def mat(name, n, k, gain=1.0):
        w[name] = bf16(rs.randn(n, k) * gain / np.sqrt(k))

    def vec(name, n, lo, hi):
        w[name] = bf16(rs.uniform(lo, hi, size=n))

    def norm(name):
        vec(name, wd, 0.6, 1.4)
        vec(name + ".b", wd, -0.2, 0.2)

    def ff(p, n, bias):
        mat(p + "gate", n, wd, 1.5)
        mat(p + "up", n, wd)
        mat(p + "down", wd, n, 1.5)
        if bias:
            vec(p + "gate.b", n, -0.5, 0.5)
            vec(p + "up.b", n, -0.5, 0.5)
            vec(p + "down.b", wd, -0.3, 0.3)

    w["embed"] = bf16(rs.randn(cfg["vocab"], wd))
    big = cfg.get("embedding", {}).get("bigram")
    if big:
        w["bigram"] = bf16(rs.randn(big["buckets"] + 1, wd))
    if cfg.get("loop"):
        mat("loop.in", wd, 2 * wd)
    mat("head", cfg["vocab"], wd, 2.0)
    norm("final.norm")
    for i, c in enumerate(cfg["layers"]):
        p, m = f"l{i}.", c["mixer"]
        norm(p + "norm1")
        if c["type"] == "mlstm":
            hd, hv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            for n, k in (("q", hd), ("k", hd), ("v", hv), ("g", hv)):
                mat(p + "mix." + n, k, wd, 2.0 if n == "q" else 1.0)
            mat(p + "mix.o", wd, hv, 1.5)
            vec(p + "mix.norm", hv, 0.5, 1.5)
            mat(p + "mix.i", m["heads"], wd, 1.5)
            mat(p + "mix.f", m["heads"], wd, 0.5)
            vec(p + "mix.i.b", m["heads"], -2.0, 1.0)
            vec(p + "mix.f.b", m["heads"], 3.0, 6.0)
        else:
            heads, dim, rot, vdim, rank = (m[n] for n in ("heads", "dim", "rot_dim", "vdim",
                                                          "kv_rank"))
            mat(p + "mix.q", heads * (dim + rot), wd, 2.0)
            mat(p + "mix.dkv", rank + rot, wd)
            vec(p + "mix.dkv.norm", rank, 0.5, 1.5)
            mat(p + "mix.uk", heads * dim, rank)
            mat(p + "mix.uv", heads * vdim, rank)
            mat(p + "mix.o", wd, heads * vdim, 1.5)
        f = c.get("mlp")
        if not f:
            continue
        norm(p + "norm2")
        if f["kind"] == "dense":
            ff(p + "mlp.", f["ff"], True)
            continue
        n = f["router"]["experts"]
        mat(p + "mlp.router", n, wd, 2.0)
        vec(p + "mlp.router.b", n, -0.5, 0.5)
        for e in range(n):
            ff(f"{p}mlp.e{e}.", f["expert"]["ff"], False)
            # experts resemble the first one, so that a choice which hangs on the last bits
            # of a row does not change the row beyond recognition
            for leaf in ("gate", "up", "down") if e else ():
                first, own = w[f"{p}mlp.e0.{leaf}"], w[f"{p}mlp.e{e}.{leaf}"]
                w[f"{p}mlp.e{e}.{leaf}"] = bf16(first + 0.25 * own)
        if f.get("shared"):
            ff(p + "mlp.shared.", f["shared"]["ff"], False)
    return w


def write_folder(folder, cfg, w):
    """config.json + model.safetensors (bf16) of a small model."""
    header, blobs, at = {}, [], 0
    for name, a in w.items():
        raw = (np.ascontiguousarray(a, dtype=np.float32).view(np.uint32) >> 16).astype("<u2").tobytes()
        header[name] = {"dtype": "BF16", "shape": list(np.shape(a)),
                        "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    head = json.dumps(header).encode()
    (folder / "config.json").write_text(json.dumps(cfg))
    with open(folder / "model.safetensors", "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head + b"".join(blobs))
