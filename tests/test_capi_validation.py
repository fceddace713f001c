"""The C-ABI refuses bad arguments on the host, before any CUDA call: these run
without a GPU.  Every refusal returns a negative fk_status and leaves a message
in fk_last_error()."""
import ctypes

import pytest

from fastkernels_b200 import _lib

L = _lib.lib
INVALID, UNSUPPORTED, WORKSPACE, ALIGNMENT = -1, -2, -3, -4
P = 0x10000          # a non-null, 16-byte aligned stand-in; never dereferenced


def err():
    return L.fk_last_error().decode()


def prefill(**kw):
    a = dict(q=P, q_stride=512, out=P, out_stride=512, lse=None, k=P, v=P, kv_stride=256,
             num_blocks=0, block_size=0, layout=0, cu_q=P, cu_k=P, bt=None, bt_stride=0,
             num_seqs=1, total_q=8, total_k=8, max_q=8, hq=4, hkv=2, d=128, scale=0.1, causal=1)
    a.update(kw)
    return L.fk_prefill_attn(a["q"], a["q_stride"], a["out"], a["out_stride"], a["lse"], a["k"],
                             a["v"], a["kv_stride"], a["num_blocks"], a["block_size"],
                             a["layout"], a["cu_q"], a["cu_k"], a["bt"], a["bt_stride"],
                             a["num_seqs"], a["total_q"], a["total_k"], a["max_q"], a["hq"],
                             a["hkv"], a["d"], a["scale"], a["causal"], None, None)


def test_prefill_refusals():
    assert prefill(num_seqs=0) == 0                      # empty batch: nothing to do
    assert prefill(total_q=0) == 0
    assert prefill(q=None) == INVALID and "null" in err()
    assert prefill(d=64) == UNSUPPORTED and "head_dim" in err()
    assert prefill(hq=5) == INVALID and "multiple" in err()
    assert prefill(q=P + 2) == ALIGNMENT
    assert prefill(q_stride=509) == ALIGNMENT
    assert prefill(q_stride=128) == INVALID and "stride" in err()
    assert prefill(num_blocks=4, block_size=64, kv_stride=64 * 2 * 128) == INVALID  # no tables
    assert prefill(num_blocks=4, block_size=48, kv_stride=48 * 2 * 128, bt=P,
                   bt_stride=4) == UNSUPPORTED and "block_size" in err()
    assert prefill(num_blocks=4, block_size=64, kv_stride=64 * 2 * 128, bt=P, bt_stride=4,
                   layout=7) == INVALID and "kv_layout" in err()
    assert prefill(total_k=0) == INVALID


def test_merge_refusals():
    def merge(**kw):
        a = dict(out=P, st=512, sh=128, lse=None, a=P, b=P, al=P, bl=P, tokens=4, heads=4, d=128)
        a.update(kw)
        return L.fk_merge_attn_states(a["out"], a["st"], a["sh"], a["lse"], a["a"], a["st"],
                                      a["sh"], a["al"], a["b"], a["st"], a["sh"], a["bl"],
                                      a["tokens"], a["heads"], a["d"], -1, None)
    assert merge(tokens=0) == 0
    assert merge(a=None) == INVALID
    assert merge(d=12) == UNSUPPORTED and "multiple of 8" in err()
    assert merge(out=P + 4) == ALIGNMENT
    assert merge(sh=100) == ALIGNMENT


def test_decode_side_refusals():
    # head_dim other than 128, GQA ratio not a power of two up to 16, odd page size
    args = lambda **kw: _attn(**kw)                        # noqa: E731
    assert _attn(d=64) == UNSUPPORTED
    assert _attn(hq=6, hkv=2) == UNSUPPORTED and "GQA" in err()
    assert _attn(block=48) == UNSUPPORTED
    assert _attn(ws=None) == WORKSPACE
    # GEMM: k not a multiple of 64, missing workspace
    assert L.fk_gemm_bf16(P, 4096, P, None, P, 4096, 8, 4096, 4000, P, 1 << 30, None,
                          None) == UNSUPPORTED and "64" in err()
    assert L.fk_gemm_bf16(P, 4096, P, None, P, 4096, 8, 4096, 4096, None, 0, None,
                          None) == WORKSPACE
    assert L.fk_gemm_bf16_static(P, 4096, P, None, P, 4096, 65, 4096, 4096, None,
                                 None) == UNSUPPORTED and "scratch" in err()


def _attn(d=128, hq=8, hkv=2, block=64, ws=P):
    return L.fk_paged_decode_attn(P, hq * d, P, hq * d, P, P, 16, block, block * hkv * d, 0, P, P,
                                  4, 2, hq, hkv, d, 0.1, 8, ws, 1 << 24, None, None)


def group_gemm(**kw):
    a = dict(x=P, xs=256, xg=0, xr=8, w=P, bias=None, y=P, ys=128, yg=0, f32=0, yf32=0, off=None,
             gather=None, rows=8, expect=8, groups=1, n=128, k=256, act=-1)
    a.update(kw)
    return L.fk_group_gemm(a["x"], a["xs"], a["xg"], a["xr"], a["w"], a["bias"], a["y"], a["ys"],
                           a["yg"], a["f32"], a["yf32"], a["off"], a["gather"], a["rows"],
                           a["expect"], a["groups"], a["n"], a["k"], a["act"], None, None)


def test_grouped_projection_refusals():
    assert group_gemm(rows=0) == 0
    assert group_gemm(w=None) == INVALID and "null" in err()
    assert group_gemm(k=252) == ALIGNMENT                       # bf16 rows of 16 bytes
    assert group_gemm(f32=1, yf32=0) == INVALID
    assert group_gemm(act=7) == INVALID and "activation" in err()
    assert group_gemm(act=0, yf32=1) == UNSUPPORTED
    assert group_gemm(gather=P) == INVALID and "row groups" in err()
    assert group_gemm(xr=7) == INVALID and "few rows" in err()
    assert group_gemm(groups=2, xg=128, yg=64, ys=256) == INVALID    # x rows too short
    assert group_gemm(groups=2, xs=512, xg=256, ys=256, yg=100) == INVALID   # overlapping y


def test_routing_refusals():
    def route(**kw):
        a = dict(z=P, zs=16, rows=4, experts=16, top=2, counts=None)
        a.update(kw)
        return L.fk_moe_route(a["z"], a["zs"], P, P, P, P, P, a["counts"], a["rows"],
                              a["experts"], a["top"], None)
    assert route(rows=0) == 0
    assert route(top=17) == INVALID
    assert route(zs=15) == INVALID
    assert route(experts=2000, zs=2000) == UNSUPPORTED
    assert L.fk_moe_route_counts(64, 16, 2) == 0 < L.fk_moe_route_counts(8192, 16, 2)
    assert route(rows=8192) == WORKSPACE
    assert L.fk_gather_rows(P, 64, 4, P, P, 4, 24, None, None) == ALIGNMENT


def test_latent_attention_refusals():
    def attn(**kw):
        a = dict(q=P, qp=576, cp=576, op=512, bs=64, rows=4, heads=16, rank=512, rot=32, splits=1,
                 ws=None, n=0)
        a.update(kw)
        return L.fk_latent_attn(a["q"], a["qp"], P, 16, a["bs"], a["cp"], P, a["op"], P, P, P, 4,
                                4, a["rows"], 1, a["heads"], a["rank"], a["rot"], 0.1,
                                a["splits"], a["ws"], a["n"], None, None)
    assert attn(rows=0) == 0
    assert attn(q=None) == INVALID
    assert attn(rank=528, op=528) == UNSUPPORTED and "rank" in err()
    assert attn(cp=520) == UNSUPPORTED and "64" in err()
    assert attn(qp=512) == INVALID
    assert attn(bs=12) == UNSUPPORTED and "block_size" in err()
    assert attn(splits=4) == WORKSPACE
    assert attn(splits=40) == INVALID
    assert L.fk_latent_attn_supported(512, 64) == 1 and L.fk_latent_attn_supported(520, 8) == 0
    for seqs, heads in ((1, 16), (64, 16), (64, 40), (300, 128)):
        assert 1 <= L.fk_latent_attn_splits(seqs, 1, heads, 512, 16384) <= 32
    assert L.fk_latent_attn_splits(1, 1, 16, 512, 100) == 1
    assert L.fk_latent_prepare(P, P, 512, 40, 0, P, P, 64, P, P, P, 64, 128, P, 64, 0, 1, 4, 4, 24,
                               16, 64, 1e-5, None, None) == INVALID    # copy over the rotated part


def test_matrix_memory_refusals():
    def portions(**kw):
        a = dict(q=P, f32=0, zs=16, heads=8, dim=64, vdim=64, cap=5.0, ws=P, n=1 << 40)
        a.update(kw)
        return L.fk_mlstm_portions(a["q"], P, P, 2048, a["f32"], P, a["zs"], P, P, 4, P, 2, P, P,
                                   P, 300, a["heads"], a["dim"], a["vdim"], a["cap"], 0.1,
                                   a["ws"], a["n"], 200, None, None)
    assert portions(q=None) == INVALID
    assert portions(zs=15) == INVALID
    assert portions(cap=0.0) == INVALID
    assert portions(dim=600) == UNSUPPORTED and portions(vdim=1100) == UNSUPPORTED
    assert portions(n=100) == WORKSPACE
    assert L.fk_mlstm_state_cols(65) == 68 and L.fk_mlstm_norm_cols(64) == 68
    need = L.fk_mlstm_workspace_floats(300, 2, 8, 64, 64)
    assert need > 4 * 8 * 64 * 64


def test_row_kernel_refusals():
    def add(**kw):
        a = dict(x=P, xo=P, a=P, ast=128, w1=P, b1=P, o1=P, w2=None, b2=None, o2=None, width=120)
        a.update(kw)
        return L.fk_add_layernorm(a["x"], a["xo"], a["a"], a["ast"], None, 0, None, 0, 0, None,
                                  None, 0, a["w1"], a["b1"], a["o1"], 128, a["w2"], a["b2"],
                                  a["o2"], 128, 0, 4, 128, a["width"], 1e-5, None, None)
    assert add(x=None) == INVALID
    assert add(b1=None) == INVALID and add(o2=P) == INVALID
    assert add(width=200) == INVALID
    assert add(ast=100) == INVALID and add(ast=130) == ALIGNMENT
    assert L.fk_embed_pair_f32(P, P, 0, 10, 0, 1, 1, P, P, 4, P, P, P, 1, P, None, 0, 4, 64, None,
                               None) == INVALID and "pair table" in err()
    assert L.fk_softcap(P, 8, 0, 2, 16, 5.0, None) == INVALID
    assert L.fk_softcap(P, 16, 0, 2, 16, 0.0, None) == INVALID
