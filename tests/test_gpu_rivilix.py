"""Rivilix on the GPU against the plain oracle: each mechanism alone, then the whole decoder
through the engine (prompts, portions, single tokens, batches, reuse of pages and slots,
greedy generation), in fp32 and bf16."""
import io
import json
import os
import subprocess

import numpy as np
import pytest
import torch

import rivilix_oracle as R

pytestmark = pytest.mark.gpu

F32, BF16 = torch.float32, torch.bfloat16
DTYPES = [F32, BF16]


def dev(a, dtype=F32):
    return torch.from_numpy(np.ascontiguousarray(a)).to("cuda", dtype)


def values(rs, *shape, dtype=F32):
    """float64 values that dtype holds exactly."""
    a = rs.randn(*shape)
    return R.bf16(a) if dtype == BF16 else a.astype(np.float32).astype(np.float64)


def close(got, want, dtype, scale=1.0):
    """fp32: 2e-5 of the values' scale; bf16: two rounding steps of it."""
    tol = (2e-5 if dtype == F32 else 1.2e-2) * scale
    np.testing.assert_allclose(got.double().cpu().numpy(), want, rtol=tol, atol=tol)


def i32(a):
    return torch.tensor(np.asarray(a), dtype=torch.int32, device="cuda")


def i64(a):
    return torch.tensor(np.asarray(a), dtype=torch.int64, device="cuda")


def padded(a, cols):
    out = np.zeros((*a.shape[:-1], cols))
    out[..., :a.shape[-1]] = a
    return out


# ------------------------------------------------------------------- row mechanisms
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [40, 320])
def test_embedding_pairs_across_portions(width, dtype):
    """Four sequences in portions cut anywhere, single tokens, a padded row; slots change
    hands without being cleared."""
    from fastkernels_b200 import ops
    rs = np.random.RandomState(width)
    vocab, buckets, mp, mc = 60, 23, 1009, 7
    stride = (width + 63) // 64 * 64
    tab, pairs = values(rs, vocab, width, dtype=dtype), values(rs, buckets + 1, width, dtype=dtype)
    td, pd = dev(padded(tab, stride), dtype), dev(padded(pairs, stride), dtype)
    last = torch.full((5,), 55, dtype=torch.int64, device="cuda")
    seqs = [rs.randint(0, vocab, size=n) for n in (30, 17, 9, 40)]
    want = [tab[s] + pairs[R.bigram_rows(s, buckets, mp, mc)] for s in seqs]
    at, slots = [0] * 4, [3, 0, 4, 3]
    st = ops.new_status("cuda")
    for batch in ([(0, 2), (1, 1), (2, 5)], [(1, 1), (0, 1)], [(0, 26), (2, 1), (1, 14)], [(0, 1)],
                  [(3, 1), (1, 1)], [(3, 38), (2, 3)], [(3, 1)]):
        ids = np.concatenate([seqs[i][at[i]:at[i] + n] for i, n in batch] + [[1]])
        pos = np.concatenate([np.arange(at[i], at[i] + n) for i, n in batch] + [[0]])
        sl = np.concatenate([[slots[i]] * n for i, n in batch] + [[-1]])
        cu = np.concatenate([[0], np.cumsum([n for _, n in batch] + [1])])
        both = torch.zeros((len(ids), 2 * stride), dtype=dtype, device="cuda")
        x = ops.embed_pair_f32(td, i64(ids), pd, mp, mc, last, i32(sl), i64(pos), i32(cu),
                               copy=both[:, stride:], status=st)
        ref = np.concatenate([want[i][at[i]:at[i] + n] for i, n in batch]
                             + [tab[1:2] + pairs[buckets:]])
        close(x[:, :width], ref, F32)
        close(both[:, stride:stride + width], ref, dtype)
        assert torch.count_nonzero(x[:, width:]) == 0 and torch.count_nonzero(both[:, :stride]) == 0
        for i, n in batch:
            at[i] += n
            assert int(last[slots[i]]) == seqs[i][at[i] - 1]
    assert int(last[1]) == 55 and int(st.item()) == 0
    x = ops.embed_pair_f32(td, i64([3, 59]))
    close(x[:, :width], tab[[3, 59]], F32)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,rows", [(40, 3), (191, 500), (1100, 37), (5000, 400), (9000, 5)])
def test_add_layernorm(width, rows, dtype):
    from fastkernels_b200 import ops
    rs = np.random.RandomState(rows)
    stride, eps, top = (width + 63) // 64 * 64, 1e-3, 3
    x = values(rs, rows, width) + 2.0
    a, b, e = (values(rs, n, width, dtype=dtype) for n in (rows, rows, rows * top))
    place = np.stack([rs.permutation(rows * top)[:top] for _ in range(rows)])
    share = rs.rand(rows, top).astype(np.float32)
    norms = [(rs.rand(width) + 0.5, rs.randn(width)) for _ in range(2)]
    nd = [tuple(dev(padded(v, stride)) for v in n) for n in norms]

    def run(full, two, **kw):
        xd = dev(padded(x, stride))
        add = dict(a=dev(padded(a, stride), dtype), b=dev(padded(b, stride), dtype),
                   experts=(dev(padded(e, stride), dtype), i32(place), dev(share))) if full else {}
        got = ops.add_layernorm(xd, width, eps, dtype, **add, norm1=nd[0],
                                norm2=nd[1] if two else None, **kw)
        s = x + (a + b + np.einsum("tj,tjw->tw", share, e[place]) if full else 0.0)
        close(got[0][:, :width], s, F32, scale=np.abs(s).max())
        for o, (w, bb) in zip(got[1:], norms if two else norms[:1]):
            close(o[:, :width], R.layer_norm(s, w, bb, eps), dtype, scale=2)
            assert torch.count_nonzero(o[:, width:]) == 0
        assert got[0] is xd
    run(True, True)
    run(False, True)
    run(True, False)
    # the sum itself, into columns of a wider row
    both = torch.full((rows, 2 * stride), 7.0, dtype=dtype, device="cuda")
    xd = dev(padded(x, stride))
    ops.add_layernorm(xd, width, eps, dtype, a=dev(padded(a, stride), dtype),
                      out1=both[:, :stride])
    close(both[:, :width], x + a, dtype)
    assert torch.all(both[:, stride:] == 7.0) and torch.count_nonzero(both[:, width:stride]) == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_softcap(dtype):
    from fastkernels_b200 import ops
    z = values(np.random.RandomState(0), 5, 333, dtype=dtype) * 20
    zd = dev(padded(z, 336), dtype)
    got = ops.softcap(zd[:, :333], 13.0)
    close(got, 13.0 * np.tanh(z / 13.0), dtype, scale=13)
    assert torch.count_nonzero(zd[:, 333:]) == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [6, 20, 65, 136, 256, 260, 512, 1000])
def test_head_norm_gate_sizes(dim, dtype):
    from fastkernels_b200 import ops
    rs = np.random.RandomState(dim)
    t, heads, eps = 21, 3, 1e-4
    o, g = values(rs, t, heads, dim), values(rs, t, heads * dim, dtype=dtype)
    w = rs.rand(heads * dim)
    out = torch.full((t, (heads * dim + 63) // 64 * 64), 5.0, dtype=dtype, device="cuda")
    gp = dev(padded(g, (heads * dim + 7) // 8 * 8), dtype)
    ops.head_norm_gate(dev(o.reshape(t, -1)), gp, dev(w), heads, dim, eps, out)
    close(out[:, :heads * dim], R.rms(o, eps).reshape(t, -1) * w * R.sigmoid(g), dtype)
    assert torch.count_nonzero(out[:, heads * dim:]) == 0


# --------------------------------------------------------------- grouped projections
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 2, 7, 9, 20, 40, 64, 65, 130, 300])
@pytest.mark.parametrize("groups,n,k", [(1, 24, 64), (5, 40, 48), (3, 272, 136), (1, 13, 2048)])
def test_column_groups(rows, groups, n, k, dtype):
    """Every group its own columns, between columns that stay as they were."""
    from fastkernels_b200 import ops
    rs = np.random.RandomState(rows + n)
    x = values(rs, rows, groups, k + 8, dtype=dtype)
    w = values(rs, groups, n, k, dtype=dtype) / 8
    bias = values(rs, n) if groups != 3 else None
    pitch = (n + 7) // 8 * 8
    want = np.einsum("tgk,gnk->tgn", x[:, :, :k], w) + (bias if bias is not None else 0)
    xd, wd = dev(x.reshape(rows, -1), dtype), dev(w, dtype)
    for f32 in (False, True):
        out = torch.full((rows, groups * pitch), 3.0, device="cuda",
                         dtype=F32 if f32 or dtype == F32 else BF16)
        ops.group_gemm(xd, wd, out=out, bias=dev(bias) if bias is not None else None,
                       x_group=k + 8, y_group=pitch, out_f32=f32)
        got = out.view(rows, groups, pitch)
        close(got[:, :, :n], want, out.dtype, scale=np.abs(want).max())
        assert torch.all(got[:, :, n:] == 3.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("act", [None, 0, 1])
@pytest.mark.parametrize("counts", [[3, 0, 1, 9], [0, 0, 0, 1], [70, 0, 129, 1, 128, 300],
                                    [1] * 200, [17, 33, 65]])
def test_row_groups(counts, act, dtype):
    """Rows between offsets, gathered or in place; groups without rows; many groups; both
    forms of the kernel at every size."""
    from fastkernels_b200 import ops
    rs = np.random.RandomState(len(counts))
    groups, rows, n, k = len(counts), sum(counts), 72, 128
    x = values(rs, 50, k, dtype=dtype)
    w = values(rs, groups, n if act is None else 2 * n, k, dtype=dtype) / 8
    source = rs.randint(0, 50, size=rows)
    off = np.concatenate([[0], np.cumsum(counts)])
    g = np.repeat(np.arange(groups), counts)
    z = np.einsum("tk,tnk->tn", x[source], w[g])
    if act is not None:
        a = z[:, :n]
        gate = R.silu(a) if act == 0 else \
            0.5 * a * (1 + np.tanh(np.sqrt(2 / np.pi) * (a + 0.044715 * a ** 3)))
        z = gate * z[:, n:]
    xd, wd, sd = dev(x, dtype), dev(w, dtype), i32(source)
    for gather in (True, False):
        xs = xd if gather else ops.gather_rows(xd, sd)
        if not gather:
            assert torch.equal(xs, xd[sd.long()])
        for expect in (1, 12, 20, 50, 1000):
            got = ops.group_gemm(xs, wd, offsets=i32(off), gather=sd if gather else None, act=act,
                                 expect_rows=expect)
            close(got, z, dtype, scale=np.abs(z).max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 37, 64, 300])
@pytest.mark.parametrize("ff,bias", [(56, True), (200, False), (333, True)])
def test_gated_feed_forward(rows, ff, bias, dtype):
    """Few and many rows; a width of the feed-forward that is no multiple of anything."""
    from fastkernels_b200.models.feedforward import GatedFeedForward
    from fastkernels_b200.models.weights import DictSource, Packer
    rs = np.random.RandomState(rows)
    width, stride = 88, 128
    w = {k[len("l0."):]: v for k, v in R.random_weights(
        R.model_config([R.memory_layer(mlp=R.dense(ff))], width=width), ff).items()
        if k.startswith("l0.mlp.")}
    m = GatedFeedForward(ff, bias)
    m.load(Packer(DictSource({n: torch.from_numpy(a) for n, a in w.items()}), "cuda", dtype, width,
                  stride), "mlp.")
    h = values(rs, rows, width, dtype=dtype)
    y, none = m.forward(dev(padded(h, stride), dtype))
    want = R.gated(h, w, "mlp.", bias)
    assert none is None and torch.count_nonzero(y[:, width:]) == 0
    close(y[:, :width], want, dtype, scale=2 * np.abs(want).max())


@pytest.mark.parametrize("rows,experts,top", [(1, 1, 1), (1, 9, 9), (5, 40, 5), (70, 7, 3),
                                              (300, 130, 8), (3000, 12, 2), (5000, 300, 6)])
def test_routing(rows, experts, top):
    from fastkernels_b200 import ops
    rs = np.random.RandomState(rows)
    z = rs.randn(rows, experts).astype(np.float32)
    z[::3, experts // 2:] = z[::3, :1]               # ties go to the lowest index
    r = ops.moe_route(dev(padded(z, experts + 3))[:, :experts], top)
    order = np.argsort(-z.astype(np.float64), axis=1, kind="stable")[:, :top]
    assert np.array_equal(r.chosen.cpu().numpy(), order)
    zc = np.take_along_axis(z.astype(np.float64), order, 1)
    e = np.exp(zc - zc.max(1, keepdims=True))
    close(r.share, e / e.sum(1, keepdims=True), F32)
    off, place, source = (t.cpu().numpy() for t in (r.offsets, r.place, r.source))
    assert np.array_equal(off, np.concatenate([[0], np.cumsum(np.bincount(order.ravel(),
                                                                         minlength=experts))]))
    assert sorted(place.ravel()) == list(range(rows * top))
    assert np.array_equal(source[place], np.repeat(np.arange(rows)[:, None], top, 1))
    assert np.all((place >= off[order]) & (place < off[order + 1]))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,experts,top,ff,shared", [(1, 6, 2, 40, None), (3, 5, 5, 24, 88),
                                                        (70, 9, 1, 130, 30), (600, 4, 2, 72, 72)])
def test_mixture_of_experts(rows, experts, top, ff, shared, dtype):
    from fastkernels_b200 import ops
    from fastkernels_b200.models.feedforward import MixtureOfExperts
    from fastkernels_b200.models.weights import DictSource, Packer
    rs = np.random.RandomState(rows)
    width, stride = 88, 128
    cfg = R.model_config([R.memory_layer(mlp=R.experts(experts, top, ff, shared))], width=width)
    w = R.random_weights(cfg, rows)
    m = MixtureOfExperts(experts, top, ff, shared)
    m.load(Packer(DictSource({n: torch.from_numpy(a) for n, a in w.items()}), "cuda", dtype, width,
                  stride), "l0.mlp.")
    h = values(rs, rows, width, dtype=dtype)
    dense, ex = m.forward(dev(padded(h, stride), dtype))
    x, _, _ = ops.add_layernorm(torch.zeros((rows, stride), device="cuda"), width, 1e-5, dtype,
                                b=dense, experts=ex)
    want = R.mixture(h, w, "l0.mlp.", cfg["layers"][0]["mlp"])
    close(x[:, :width], want, dtype, scale=2 * np.abs(want).max())
    assert torch.count_nonzero(x[:, width:]) == 0


# ------------------------------------------------------------------ latent attention
class Paged:
    """Sequences in shuffled pages of a pool."""

    def __init__(self, rs, lens, page, row, dtype):
        self.page = page
        n = [(x + page - 1) // page for x in lens]
        perm = rs.permutation(sum(n) + 3)
        self.tables = np.full((len(lens), max(n)), -1)
        at = 0
        for i, c in enumerate(n):
            self.tables[i, :c] = perm[at:at + c]
            at += c
        self.pool = torch.full((sum(n) + 3, page, 1, row), 9.0, dtype=dtype, device="cuda")

    def slots(self, i, a, b):
        p = np.arange(a, b)
        return self.tables[i, p // self.page] * self.page + p % self.page


LATENT_SIZES = [(5, 24, 8, 20, 40), (1, 16, 16, 24, 16), (16, 64, 32, 64, 256), (19, 15, 2, 33, 130),
                (3, 120, 40, 136, 200), (40, 32, 64, 16, 512)]


def latent_module(sizes, dtype, yarn=(4.0, 60, 8.0, 0.5), scale=0.3, seed=0, far=None):
    from fastkernels_b200 import ops
    from fastkernels_b200.models.mixers import LatentAttention, Yarn, rope_table
    from fastkernels_b200.models.weights import DictSource, Packer
    h, dim, rot, vdim, rank = sizes
    cfg = R.model_config([R.latent_layer(h, dim, rot, vdim, rank, scale, 900.0, yarn)], width=96)
    w = R.random_weights(cfg, seed)
    att = LatentAttention(h, dim, rot, vdim, rank, scale, 900.0, Yarn(*yarn), 0, 1e-4, dtype)
    p = Packer(DictSource({n: torch.from_numpy(a) for n, a in w.items()}), "cuda", dtype, 96, 128)
    rows = att.load(p, "l0.mix.")
    att.cos_sin = rope_table(900, rot, 900.0, "cuda", Yarn(*yarn))
    att.status = ops.new_status("cuda")
    return cfg["layers"][0]["mixer"], w, att, rows


def project(att, rows, h, dtype):
    """Packed projection rows of h as the model makes them, and their columns."""
    return pack(att, {n: h @ rows[n].double().cpu().numpy().T for n in att.sections}, dtype)


def pack(att, sections, dtype):
    at, cols = 0, {}
    parts = []
    for n, c in att.sections.items():
        z = R.bf16(sections[n]) if dtype == BF16 else sections[n]
        size = (c + 7) // 8 * 8
        parts.append(padded(z, size))
        cols[n] = (at, at + c)
        at += size
    z = dev(np.concatenate(parts + [np.full((len(parts[0]), 16), 4.0)], 1), dtype)
    return {n: z[:, a:b] for n, (a, b) in cols.items()}


def run_latent(att, cols, paged, batch, decode=False, graph_cols=None):
    """batch: [(sequence, first position, count)] over the rows of cols."""
    from fastkernels_b200.infra import context
    cu = np.concatenate([[0], np.cumsum([n for _, _, n in batch])])
    kv = np.array([a + n for _, a, n in batch])
    span = context.SpanBatch(
        i32(np.concatenate([paged.slots(i, a, a + n) for i, a, n in batch])),
        i32(paged.tables[[i for i, _, _ in batch]]), i32(kv), i32(cu),
        i32(np.concatenate([[0], np.cumsum(kv)])), max(n for _, _, n in batch), int(kv.max()),
        int(kv.sum()))
    context.set_context(not decode, spans=[span])
    try:
        pos = np.concatenate([np.arange(a, a + n) for _, a, n in batch])
        return att.forward(None, cols, i64(pos), 0)
    finally:
        context.reset_context()


def plain_heads(cfg, w, h):
    """Attention output per head, ahead of the output projection."""
    p = {n: a for n, a in w.items() if n.startswith("l0.mix.")}
    width = cfg["heads"] * cfg["vdim"]
    return R.latent_mixer(h, {**p, "l0.mix.o": np.eye(width)}, "l0.mix.", cfg, 1e-4)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", LATENT_SIZES)
def test_latent_attention_portions_and_tokens(sizes, dtype):
    """Three sequences in one batch: whole, in portions (expanded and absorbed), token by
    token; pages shuffled; rounding aside all the same."""
    cfg, w, att, rows = latent_module(sizes, dtype, scale=1.2 / np.sqrt(sizes[1] + sizes[2]))
    rs = np.random.RandomState(3)
    lens = [150, 33, 71]
    hs = [values(rs, n, 96, dtype=dtype) for n in lens]
    want = [plain_heads(cfg, w, h) for h in hs]
    vp, vd, heads = att.v_pitch, cfg["vdim"], cfg["heads"]
    for cuts in ([[150], [33], [71]], [[2, 90, 58], [1, 30, 2], [40, 2, 29]],
                 [[149, 1], [31, 1, 1], [70, 1]]):
        paged = Paged(rs, lens, 16, att.row, dtype)
        att.caches = [paged.pool]
        at = [0, 0, 0]
        for step in range(3):
            batch = [(i, at[i], cuts[i][step]) for i in range(3) if step < len(cuts[i])]
            if not batch:
                continue
            cols = project(att, rows, np.concatenate([hs[i][a:a + n] for i, a, n in batch]), dtype)
            out = run_latent(att, cols, paged, batch,
                             decode=all(n == 1 and a > 0 for _, a, n in batch))
            assert torch.count_nonzero(out[:, heads * vp:]) == 0
            got = out[:, :heads * vp].view(-1, heads, vp)
            assert torch.count_nonzero(got[:, :, vd:]) == 0
            got = got[:, :, :vd].reshape(len(got), -1)
            row = 0
            for i, a, n in batch:
                close(got[row:row + n], want[i][a:a + n], dtype, scale=2 * np.abs(want[i]).max())
                row += n
                at[i] += n
    assert int(att.status.item()) == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_key_that_stands_out_everywhere(dtype):
    """One early key per trial carries the whole softmax for all later queries: at page
    borders, tile borders, the first and the last place, in prompts and in decoding."""
    sizes = heads, dim, rot, vdim, rank = 4, 32, 16, 24, 48
    cfg, w, att, _ = latent_module(sizes, dtype, scale=0.2, seed=5)
    rs = np.random.RandomState(1)
    n, vp = 200, att.v_pitch

    def of_heads(o):
        return o[:, :heads * vp].view(-1, heads, vp)[:, :, :vdim].reshape(len(o), -1)
    for place in (0, 1, 15, 16, 63, 64, 65, 127, 128, 190, 198):
        q, z = rs.randn(n, heads, dim + rot), rs.randn(n, rank + rot) * 0.5
        key = w["l0.mix.uk"] @ (R.rms(z[place, :rank], 1e-4) * w["l0.mix.dkv.norm"])
        key = key.reshape(heads, dim)
        q[:, :, :dim] += 14.0 * key / np.linalg.norm(key, axis=1, keepdims=True)
        q, z = (R.bf16(a) if dtype == BF16 else a for a in (q, z))
        want = R.latent_attend(q, z, w, "l0.mix.", cfg, 1e-4)
        lat = R.rms(z[place, :rank], 1e-4) * w["l0.mix.dkv.norm"]
        assert np.corrcoef(want[-1], w["l0.mix.uv"] @ lat)[0, 1] > 0.9     # it does stand out
        paged = Paged(rs, [n], 16, att.row, dtype)
        att.caches = [paged.pool]
        q = np.concatenate([q, np.zeros((n, heads, att.q_pitch - dim - rot))], 2)
        cols = pack(att, {"q": q.reshape(n, -1), "dkv": z}, dtype)
        out = run_latent(att, {k: v[:191] for k, v in cols.items()}, paged, [(0, 0, 191)])
        close(of_heads(out), want[:191], dtype, scale=2 * np.abs(want).max())
        for t in range(191, n):
            o = run_latent(att, {k: v[t:t + 1] for k, v in cols.items()}, paged, [(0, t, 1)],
                           decode=True)
            close(of_heads(o), want[t:t + 1], dtype, scale=2 * np.abs(want).max())
    assert int(att.status.item()) == 0


@pytest.mark.parametrize("heads,rank,rot", [(1, 16, 2), (16, 512, 64), (8, 128, 16), (33, 256, 32),
                                            (128, 512, 64), (5, 100, 10)])
def test_absorbed_attention_and_key_ranges(heads, rank, rot):
    """Many ranges of keys per row and none; a sequence without keys; long and short ones
    together."""
    from fastkernels_b200 import ops
    rs = np.random.RandomState(heads)
    lens = [700, 1, 0, 64, 65, 333]
    row = (rank + rot + 63) // 64 * 64
    paged = Paged(rs, [max(n, 1) for n in lens], 64, row, BF16)
    keys = []
    for i, n in enumerate(lens):
        c = padded(R.bf16(rs.randn(n, rank + rot)), row)
        keys.append(c)
        if n:
            paged.pool.view(-1, row)[torch.from_numpy(paged.slots(i, 0, n)).cuda()] = dev(c, BF16)
    q = padded(R.bf16(rs.randn(len(lens), heads, rank + rot)), row)
    scale = 2.0 / np.sqrt(rank + rot)
    want = np.zeros((len(lens), heads, rank))
    for i, n in enumerate(lens):
        if n:
            s = q[i] @ keys[i].T * scale
            s = np.exp(s - s.max(-1, keepdims=True))
            want[i] = (s / s.sum(-1, keepdims=True)) @ keys[i][:, :rank]
    args = (dev(q, BF16), paged.pool, i32(np.arange(len(lens) + 1)), i32(lens),
            i32(paged.tables), 1)
    st = ops.new_status("cuda")
    for max_keys in (64, 700, 100000):
        got = ops.latent_attn(*args, max_keys, rank, rot, scale, status=st)
        close(got[:, :, :rank], want, BF16, scale=np.abs(want).max())
    assert int(st.item()) == 0


def test_softmax_weights_of_latent_attention_keep_sixteen_bits():
    """Weights that bf16 cannot hold, with values of both signs whose sum nearly cancels."""
    from fastkernels_b200 import ops
    rs = np.random.RandomState(0)
    n, rank = 640, 64
    c = R.bf16(rs.randn(n, rank) * 0.3)
    c[:, ::2] = np.where(np.arange(n) % 3 == 0, 1.0, -0.5)[:, None]
    q = R.bf16(rs.randn(1, 1, rank) * 0.3)
    s = (c @ q[0, 0]) * 0.2
    p = np.exp(s - s.max())
    want = (p / p.sum()) @ c
    got = ops.latent_attn(dev(q, BF16), dev(c, BF16).view(-1, 64, 1, rank), i32([0, 1]), i32([n]),
                          i32([np.arange(n // 64)]), 1, n, rank, 0, 0.2)
    got = got[0, 0].double().cpu().numpy()
    assert np.abs(got - want)[::2].max() <= 2.0 ** -8 * np.abs(want[::2]).max() + 1e-5


# --------------------------------------------------------------------- matrix memory
MEMORY_SIZES = [(3, 20, 28), (1, 9, 7), (2, 64, 128), (2, 128, 64), (1, 264, 40), (2, 48, 200),
                (5, 33, 65), (1, 256, 260)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim", MEMORY_SIZES)
def test_matrix_memory_portions_and_tokens(heads, dim, vdim, dtype):
    """Sequences of unequal length in portions of 1 to 257 tokens, in blocks and one by
    one, steps in between; slots start with what others left; a padded row."""
    from fastkernels_b200 import ops
    rs = np.random.RandomState(dim)
    cap, eps, total, scale = 6.0, 1e-4, 400, dim ** -0.5
    widths = {"q": heads * dim, "k": heads * dim, "v": heads * vdim, "g": heads * vdim}
    offs, at = {}, 0
    for n, c in widths.items():
        offs[n] = at
        at += (c + 7) // 8 * 8
    rows = [values(rs, total, at, dtype=dtype) for _ in range(3)]
    zs = [np.concatenate([rs.randn(total, heads) * 3 - 1, rs.randn(total, heads) * 2 + 5], 1)
          .astype(np.float32).astype(np.float64) for _ in range(3)]
    norm = rs.rand(heads * vdim) + 0.5
    want = []
    for x, z in zip(rows, zs):
        c = {n: x[:, offs[n]:offs[n] + widths[n]] for n in widths}
        i, f = R.mlstm_gates(z[:, :heads], z[:, heads:], cap)
        o, s = R.mlstm_memory(c["q"].reshape(total, heads, dim) * scale,
                              c["k"].reshape(total, heads, dim),
                              c["v"].reshape(total, heads, vdim), i, f)
        y = R.rms(o, eps).reshape(total, -1) * norm * R.sigmoid(c["g"])
        want.append((o.reshape(total, -1), y, s))
    big = max(np.abs(w[0]).max() for w in want)
    shapes = ops.mlstm_state_shapes(5, heads, dim, vdim)
    S, N = (torch.full(s, 3.0, device="cuda") for s in shapes)     # must not leak in
    slots, at = [4, 0, 2], [0, 0, 0]
    st = ops.new_status("cuda")
    pitch = (heads * vdim + 63) // 64 * 64

    def run(portions, chunked=True, step=False):
        z = np.concatenate([rows[i][at[i]:at[i] + n] for i, n in portions] + [rows[0][:1]])
        gz = np.concatenate([zs[i][at[i]:at[i] + n] for i, n in portions] + [zs[0][:1]])
        cu = np.concatenate([[0], np.cumsum([n for _, n in portions] + [1])])
        pos = np.concatenate([np.arange(at[i], at[i] + n) for i, n in portions] + [[0]])
        sl = np.concatenate([[slots[i]] * n for i, n in portions] + [[-1]])
        zd = dev(z, dtype)
        col = {n: zd[:, offs[n]:offs[n] + widths[n]] for n in widths}
        out = torch.full((len(z), pitch), 9.0, dtype=dtype, device="cuda")
        if step:
            ops.mlstm_step(col["q"], col["k"], col["v"], dev(gz), col["g"], dev(norm), S, N,
                           i32(sl), i64(pos), heads, dim, vdim, cap, scale, eps, out, status=st)
        else:
            o = ops.mlstm_portions(col["q"], col["k"], col["v"], dev(gz), S, N, i32(cu), i32(sl),
                                   i64(pos), heads, dim, vdim, cap, scale,
                                   max(n for _, n in portions), chunked=chunked, status=st)
            ops.head_norm_gate(o, col["g"], dev(norm), heads, vdim, eps, out)
        row = 0
        for i, n in portions:
            if not step:
                # sums of both signs over their absolute value, the denominator, amplify
                # rounding where the latter is small
                got = o[row:row + n].double().cpu().numpy()
                ref = want[i][0][at[i]:at[i] + n]
                err = np.abs(got - ref) / (np.abs(ref).max(1, keepdims=True) + 0.05 * big)
                assert err.max() < (3e-4 if dtype == F32 else 2e-3), err.max()
            close(out[row:row + n, :heads * vdim], want[i][1][at[i]:at[i] + n], dtype,
                  scale=30 if dtype == F32 else 3)
            row += n
            at[i] += n
        assert torch.count_nonzero(out[:, heads * vdim:]) == 0

    run([(0, 1), (1, 70)])
    run([(0, 2), (2, 63)])
    run([(2, 1), (0, 64), (1, 1)])
    run([(0, 1), (1, 1), (2, 1)], step=True)
    run([(0, 129), (2, 2)])
    run([(1, 257), (2, 5)])
    run([(2, 17), (0, 9)], chunked=False)
    for _ in range(4):
        run([(0, 1), (2, 1)], step=True)
    run([(0, 2), (1, 2)])
    run([(2, 128), (0, 127)])
    run([(1, 60), (2, 100), (0, 45)])
    while at[0] < total or at[1] < total:
        run([(i, 1) for i in (0, 1) if at[i] < total], step=True)
    assert int(st.item()) == 0
    for i in (0, 1):
        s, n, m = want[i][2]
        top = np.abs(s).max()
        np.testing.assert_allclose(S[slots[i], :, :, :vdim].double().cpu().numpy(), s,
                                   atol=(3e-5 if dtype == F32 else 3e-4) * top)
        np.testing.assert_allclose(N[slots[i], :, :dim].double().cpu().numpy(), n,
                                   atol=(3e-5 if dtype == F32 else 3e-4) * np.abs(n).max())
        close(N[slots[i], :, dim], m, F32, scale=10)
    for free in (1, 3):
        assert torch.all(S[free] == 3.0) and torch.all(N[free] == 3.0)


@pytest.mark.parametrize("chunked", [False, True])
def test_memory_recalls_a_far_token(chunked):
    """One token with an open input gate, then hundreds with a closed one and hardly any
    forgetting: it is still what a matching query reads, wherever the portions were cut."""
    from fastkernels_b200 import ops
    rs = np.random.RandomState(2)
    t, dim, vdim, cap = 700, 32, 48, 10.0
    k, v = R.bf16(rs.randn(t, dim) * 0.3), R.bf16(rs.randn(t, vdim))
    q = R.bf16(rs.randn(t, dim) * 0.1)
    for place in (0, 1, 64, 127, 128, 129, 255, 300):
        q[-1] = k[place]
        zi = np.full((t, 1), -12.0)
        zi[place] = 4.0
        z = np.concatenate([zi, np.full((t, 1), 15.0)], 1)
        i, f = R.mlstm_gates(z[:, :1], z[:, 1:], cap)
        want, _ = R.mlstm_memory(q[:, None], k[:, None], v[:, None], i, f)
        assert np.corrcoef(want[-1, 0], v[place])[0, 1] > 0.95
        x = dev(np.concatenate([q, k, v], 1), BF16)
        for cuts in ([700], [place + 1, 699 - place], [128, 1, 2, 568, 1]):
            state = [torch.zeros(s, device="cuda") for s in ops.mlstm_state_shapes(1, 1, dim, vdim)]
            at = 0
            for n in cuts:
                o = ops.mlstm_portions(
                    x[at:at + n, :dim], x[at:at + n, dim:2 * dim], x[at:at + n, 2 * dim:],
                    dev(z[at:at + n]), *state, i32([0, n]), i32([0] * n),
                    i64(np.arange(at, at + n)), 1, dim, vdim, cap, 1.0, n, chunked=chunked)
                at += n
            close(o[-1:], want[-1:, 0], F32, scale=30 * np.abs(want[-1]).max())


# ------------------------------------------------------------------- the whole decoder
MODELS = R.MODELS
_CACHE = {}


def model(name):
    if name not in _CACHE:
        cfg = MODELS[name]
        w = R.random_weights(cfg, seed=len(name))
        rs = np.random.RandomState(11)
        seqs = [rs.randint(0, cfg["vocab"], size=n) for n in (140, 61, 23, 1, 2)]
        _CACHE[name] = (cfg, w, seqs, [R.forward(s, w, cfg) for s in seqs])
    return _CACHE[name]


def engine(name, dtype, max_seqs=6, max_len=200, pages=None, block=16, graphs=()):
    from fastkernels_b200.engine import DecodeEngine
    from fastkernels_b200.models import registry
    from fastkernels_b200.models.weights import DictSource
    cfg, w, _, _ = model(name)
    source = DictSource({n: torch.from_numpy(np.asarray(a)) for n, a in w.items()})
    config = registry._module("Rivilix").config_from_json(cfg, source, dtype)
    config.kv_block_size = block
    eng = DecodeEngine(config, max_num_seqs=max_seqs, max_model_len=max_len,
                       num_kv_blocks=pages or 120, init_scale=None)
    eng.load_weights(source)
    if graphs:
        eng.capture_cudagraph(graphs)
    return eng


class Errors:
    """Root mean square error per position, relative to the logits' own size.  A row whose
    routing is a close call may take another expert in bf16: few positions may be far off
    there, none in fp32."""

    def __init__(self, dtype):
        self.dtype, self.all = dtype, []

    def add(self, got, want):
        d = got.double().numpy() - want
        e = np.sqrt(np.mean(d ** 2, axis=1)) / np.sqrt(np.mean(want ** 2))
        self.all.append(e)
        if self.dtype == F32:
            assert e.max() < 1e-4, (e.max(), int(e.argmax()))

    def check(self):
        e = np.concatenate(self.all)
        if self.dtype == BF16:
            assert np.mean(e > 0.1) <= 0.08 and np.median(e) < 0.04, \
                (np.mean(e > 0.1), np.median(e), e.max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(MODELS))
def test_whole_prompts_alone_and_together(name, dtype):
    _, _, seqs, want = model(name)
    eng, err = engine(name, dtype), Errors(dtype)
    for s, w in zip(seqs, want):
        q = eng.open_sequence()
        err.add(eng.feed([(q, s)], [range(len(s))])[0], w)
        eng.finish(q)
    # all of them in one batch of unequal prompts
    live = [eng.open_sequence() for _ in seqs]
    for g, w in zip(eng.feed(list(zip(live, seqs)), [range(len(s)) for s in seqs]), want):
        err.add(g, w)
    err.check()
    assert eng.device_status() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("graphs", [(), (1, 3)])
@pytest.mark.parametrize("name", sorted(MODELS))
def test_token_by_token_equals_the_prompt(name, graphs, dtype):
    """From the first token on, eagerly and under CUDA graphs (with padded rows)."""
    _, _, seqs, want = model(name)
    eng, err = engine(name, dtype, graphs=graphs), Errors(dtype)
    live = [eng.open_sequence() for _ in range(2)]
    for t in range(len(seqs[0])):
        batch = [i for i in range(2) if t < len(seqs[i])]
        out = eng.feed([(live[i], seqs[i][t:t + 1]) for i in batch])
        for i, g in zip(batch, out):
            err.add(g, want[i][t:t + 1])
    err.check()
    assert eng.device_status() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(MODELS))
def test_portions_of_many_sizes_mixed_with_single_tokens(name, dtype):
    """Sequences advance at their own pace, in one batch, in portions of 1 to 50 tokens
    cut anywhere; finished ones leave and are started again in other pages and slots."""
    _, _, seqs, want = model(name)
    # pages for little more than what is live, so that they are used again and again
    eng, err = engine(name, dtype, max_seqs=3, pages=26, graphs=(1, 2)), Errors(dtype)
    rs = np.random.RandomState(2)
    live, done, started = {}, 0, 0
    slots = set()
    while done < 9:
        while len(live) < 3:
            live[started] = [started % len(seqs), eng.open_sequence(), 0]
            slots.add((started % len(seqs), live[started][1].state_slot))
            started += 1
        pick = [r for r in live if rs.rand() < 0.7] or [next(iter(live))]
        entries, places = [], []
        for r in pick:
            i, q, at = live[r]
            n = min(int(rs.choice([1, 1, 2, 3, 5, 16, 17, 50])), len(seqs[i]) - at)
            entries.append((q, seqs[i][at:at + n]))
            places.append((r, i, at, n))
        out = eng.feed(entries, [range(n) for _, _, _, n in places])
        for g, (r, i, at, n) in zip(out, places):
            err.add(g, want[i][at:at + n])
            live[r][2] += n
            if live[r][2] == len(seqs[i]):
                eng.finish(live.pop(r)[1])
                done += 1
    err.check()
    assert len(slots) > len(seqs)            # sequences came back in other slots
    for r in list(live):
        eng.finish(live.pop(r)[1])
    assert all(sorted(b.free) == list(range(26)) for b in eng.span_blocks)
    assert sorted(eng.state_slots.free) == [0, 1, 2] and eng.device_status() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["plain", "loop"])
def test_two_token_portions_and_first_tokens(name, dtype):
    _, _, seqs, want = model(name)
    eng, err = engine(name, dtype, graphs=(1,)), Errors(dtype)
    for first in (1, 2, 3):
        q, at = eng.open_sequence(), 0
        while at < 61:
            n = min(first if at == 0 else 2, 61 - at)
            out = eng.feed([(q, seqs[1][at:at + n])], [range(n)])[0]
            err.add(out, want[1][at:at + n])
            at += n
        eng.finish(q)
    err.check()


def test_other_sequences_do_not_change_a_result():
    _, _, seqs, _ = model("plain")
    eng = engine("plain", BF16)
    a = eng.open_sequence()
    alone = eng.feed([(a, seqs[1])], [range(61)])[0]
    others = [eng.open_sequence() for _ in range(3)]
    b = eng.open_sequence()
    together = eng.feed([(others[0], seqs[0]), (b, seqs[1]), (others[1], seqs[2])],
                        [[0], range(61), [0]])[1]
    assert ((alone - together).abs().amax(1) > 0.1).float().mean() < 0.05


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("graphs", [(), (2, 4)])
def test_greedy_generation_through_the_scheduler(graphs, dtype):
    """prefill (whole and in chunks) + step: every token is the oracle's arg-max, or a near
    tie of its logits."""
    cfg, w, seqs, _ = model("loop")
    prompts = [seqs[0][:30], seqs[1][:9], seqs[2][:1]]
    for chunk_tokens in (None, 13):
        eng = engine("loop", dtype, graphs=graphs)
        first = eng.prefill([p.tolist() for p in prompts], chunk_tokens=chunk_tokens)
        toks = [first] + [eng.step() for _ in range(50)]
        gaps = []
        for i, p in enumerate(prompts):
            out = [int(t[i]) for t in toks]
            assert out == eng.seqs[i].output
            lg = R.forward(np.concatenate([p, out[:-1]]), w, cfg)[len(p) - 1:]
            gaps.append((lg.max(1) - lg[np.arange(len(out)), out]) / lg.std())
        gaps = np.concatenate(gaps)
        if dtype == F32:
            assert gaps.max() <= 1e-4
        else:
            assert np.mean(gaps > 0.15) < 0.04, gaps
        assert eng.device_status() == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    """300 decoded tokens in one sequence (teacher-forced)."""
    cfg, w, _, _ = model("plain")
    s = np.random.RandomState(4).randint(0, cfg["vocab"], size=320)
    want = R.forward(s, w, cfg)
    eng, err = engine("plain", dtype, max_len=400, graphs=(1,)), Errors(dtype)
    q = eng.open_sequence()
    err.add(eng.feed([(q, s[:20])], [range(20)])[0], want[:20])
    for t in range(20, 320):
        g = eng.feed([(q, s[t:t + 1])])[0]
        if t % 7 == 0 or t > 310:
            err.add(g, want[t:t + 1])
    err.check()
    assert eng.device_status() == 0


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_runner_end_to_end(tmp_path, dtype):
    """bin/trace_run as a process: folder in, logits files out."""
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg, w, seqs, want = model("plain")
    (tmp_path / "m").mkdir()
    (tmp_path / "o").mkdir()
    R.write_folder(tmp_path / "m", cfg, w)
    s = seqs[1].tolist()
    steps, at = [], 0
    for n in (30, 2, 1, 25, 1, 1, 1):
        steps.append({"step": len(steps), "entries": [{"id": "x", "tokens": s[at:at + n],
                                                       "want": list(range(n))}], "end": []})
        at += n
    steps[-1]["end"] = ["x"]
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path / "m"),
                        "--dtype", dtype, "--out", str(tmp_path / "o"), "--max-tokens", "61"],
                       input="\n".join(json.dumps(x) for x in steps) + "\n", text=True,
                       capture_output=True, timeout=280)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == \
        [f"done {i}" for i in range(7)]
    got = np.concatenate([np.fromfile(tmp_path / "o" / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"])
                          for i in range(7)])
    err = Errors(getattr(torch, dtype))
    err.add(torch.from_numpy(got), want[1])
    err.check()


def test_generate_command_line(tmp_path):
    from fastkernels_b200 import generate
    cfg, w, seqs, _ = model("plain")
    R.write_folder(tmp_path, cfg, w)
    out = io.StringIO()
    prompts = [seqs[1][:40].tolist(), seqs[2].tolist()]
    args = ["--model", str(tmp_path), "--max-new-tokens", "12", "--dtype", "float32"]
    for p in prompts:
        args += ["--prompt", ",".join(map(str, p))]
    assert generate.main(args, stdout=out) == 0
    for p, line in zip(prompts, out.getvalue().splitlines()):
        got = [int(t) for t in line.split(",")]
        lg = R.forward(np.array(p + got[:-1]), w, cfg)[len(p) - 1:]
        assert len(got) == 12
        assert (lg.max(1) - lg[np.arange(12), got]).max() <= 1e-4 * lg.std()
