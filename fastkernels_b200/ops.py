"""Tensor-level wrappers over the C-ABI: take torch CUDA tensors, pass raw
pointers / sizes / strides and the current CUDA stream to libfk_b200.so.

torch is only the owner of device memory and streams here; every wrapper fails
loudly (FkError) instead of falling back to a torch implementation, and no
wrapper calls a library kernel.

Kernels report device-side anomalies (a slot, page or position out of range, a
bounded wait that ran out) by OR-ing fk_device_status bits into an int32 device
word.  A wrapper called without `status=` uses the per-device word of
`default_status`, so a caller that does not thread a status tensor through its
modules can still read one word per device after a step.
"""
from __future__ import annotations

import functools

import torch

from . import _lib
from ._lib import check, lib

BF16 = torch.bfloat16


def _stream() -> int:
    return torch.cuda.current_stream().cuda_stream


def _ptr(t: torch.Tensor | None) -> int | None:
    return None if t is None else t.data_ptr()


def _need(t: torch.Tensor, dtype, name: str) -> None:
    if not t.is_cuda:
        raise _lib.FkError(f"{name} must be a CUDA tensor (no CPU path exists)")
    if t.dtype != dtype:
        raise _lib.FkError(f"{name} must be {dtype}, got {t.dtype}")


def new_status(device) -> torch.Tensor:
    """One int32 device word the kernels OR their fk_device_status bits into."""
    return torch.zeros(1, dtype=torch.int32, device=device)


_DEFAULT_STATUS: dict = {}


def default_status(device=None) -> torch.Tensor:
    """The status word (one per device, made on first use) that wrappers called
    without `status=` hand to their kernels."""
    key = torch.device("cuda", torch.cuda.current_device()) if device is None \
        else torch.device(device)
    if key.index is None:
        key = torch.device("cuda", torch.cuda.current_device())
    st = _DEFAULT_STATUS.get(key)
    if st is None:
        st = _DEFAULT_STATUS[key] = new_status(key)
    return st


def _status_ptr(status, like: torch.Tensor) -> int:
    return (status if status is not None else default_status(like.device)).data_ptr()


# --------------------------------------------------------------------------- store
def store_kvcache(key, value, k_cache, v_cache, slot_mapping, status=None) -> None:
    """cache.view(-1, Hkv*D)[slot] = key[i] / value[i] for slot >= 0 (bit-exact)."""
    _need(key, k_cache.dtype, "key")
    _need(value, v_cache.dtype, "value")
    if key.element_size() != 2:
        raise _lib.FkError("store_kvcache moves 16-bit elements")
    n = key.shape[0]
    row = key[0].numel() if n else int(k_cache.shape[-1] * k_cache.shape[-2])
    if n and (key.stride(-1) != 1 or (key.dim() == 3 and key.stride(1) != key.shape[2])):
        raise _lib.FkError("key rows must be dense")
    if n and (value.stride(-1) != 1 or (value.dim() == 3 and value.stride(1) != value.shape[2])):
        raise _lib.FkError("value rows must be dense")
    if not (k_cache.is_contiguous() and v_cache.is_contiguous()):
        raise _lib.FkError("caches must be contiguous")
    if slot_mapping.dtype not in (torch.int32, torch.int64):
        raise _lib.FkError("slot_mapping must be int32 or int64")
    num_slots = k_cache.numel() // row
    check(lib.fk_store_kvcache(
        _ptr(key), _ptr(value), _ptr(k_cache), _ptr(v_cache), _ptr(slot_mapping),
        int(slot_mapping.dtype == torch.int64), n, row,
        key.stride(0) if n else row, value.stride(0) if n else row, num_slots,
        _status_ptr(status, key), _stream()), "fk_store_kvcache")


def store_kvcache_hnd(key, value, k_cache, v_cache, slot_mapping, status=None) -> None:
    """HND pool [blocks, Hkv, page, D]: head h of token i goes to
    [slot // page, h, slot % page, :] (bit-exact)."""
    _need(key, k_cache.dtype, "key")
    _need(value, v_cache.dtype, "value")
    n = key.shape[0]
    nb, hkv, page, d = k_cache.shape
    if n and (key.stride(-1) != 1 or key.stride(1) != d or value.stride(-1) != 1
              or value.stride(1) != d):
        raise _lib.FkError("key/value heads must be dense")
    if not (k_cache.is_contiguous() and v_cache.is_contiguous()):
        raise _lib.FkError("caches must be contiguous")
    if slot_mapping.dtype not in (torch.int32, torch.int64):
        raise _lib.FkError("slot_mapping must be int32 or int64")
    check(lib.fk_store_kvcache_hnd(
        _ptr(key), _ptr(value), _ptr(k_cache), _ptr(v_cache), _ptr(slot_mapping),
        int(slot_mapping.dtype == torch.int64), n, hkv, d,
        key.stride(0) if n else hkv * d, value.stride(0) if n else hkv * d, page, nb,
        _status_ptr(status, key), _stream()), "fk_store_kvcache_hnd")


# ----------------------------------------------------------------------- attention
def attn_workspace_bytes(batch, num_q_heads, head_dim, max_splits) -> int:
    return int(lib.fk_paged_decode_attn_workspace_bytes(batch, num_q_heads, head_dim,
                                                        max_splits))


def max_splits_for(max_seq_len: int, floor: int = 16) -> int:
    """Splits needed so the smallest split (128 tokens) can cover max_seq_len,
    capped: larger contexts simply use proportionally larger splits."""
    return max(1, min(64, max(floor, (max_seq_len + 127) // 128)))


def paged_decode_attn_plan(context_lens, block_tables, block_size, num_q_heads, num_kv_heads,
                           head_dim, workspace, max_splits, status=None) -> None:
    """Compute the split-KV schedule of a decode step once; layers then call
    paged_decode_attn(..., planned=True) with the same workspace."""
    _need(context_lens, torch.int32, "context_lens")
    _need(block_tables, torch.int32, "block_tables")
    b = context_lens.shape[0]
    check(lib.fk_paged_decode_attn_plan(
        _ptr(context_lens), _ptr(block_tables), block_tables.stride(0) if b else 1,
        block_size, b, num_q_heads, num_kv_heads, head_dim, int(max_splits),
        _ptr(workspace), workspace.numel() * workspace.element_size(),
        _status_ptr(status, context_lens), _stream()), "fk_paged_decode_attn_plan")


def paged_decode_attn(q, k_cache, v_cache, context_lens, block_tables, softmax_scale,
                      workspace, max_splits, out=None, status=None, planned=False,
                      kv_layout="NHD", split_weights=False):
    """out[i,h] = softmax(scale q[i,h] K_i^T) V_i over the paged cache:
    NHD [blocks, block, Hkv, D] or HND [blocks, Hkv, block, D].  split_weights: the
    fp32 weights enter P V as two bf16 parts instead of one."""
    _need(q, BF16, "q")
    _need(k_cache, BF16, "k_cache")
    _need(v_cache, BF16, "v_cache")
    _need(context_lens, torch.int32, "context_lens")
    _need(block_tables, torch.int32, "block_tables")
    b, hq, d = q.shape
    if kv_layout == "NHD":
        nb, bs, hkv, d2 = k_cache.shape
        dense = (hkv * d, d, 1)
    elif kv_layout == "HND":
        nb, hkv, bs, d2 = k_cache.shape
        dense = (bs * d, d, 1)
    else:
        raise _lib.FkError("kv_layout must be 'NHD' or 'HND'")
    if d2 != d or v_cache.shape != k_cache.shape:
        raise _lib.FkError("cache shape mismatch")
    if q.stride(2) != 1 or q.stride(1) != d:
        raise _lib.FkError("q heads must be contiguous")
    if k_cache.stride()[1:] != dense or v_cache.stride() != k_cache.stride():
        raise _lib.FkError("caches must be dense within a block")
    if block_tables.stride(1) != 1:
        raise _lib.FkError("block_tables rows must be dense")
    if out is None:
        out = torch.empty((b, hq, d), dtype=BF16, device=q.device)
    fn = lib.fk_paged_decode_attn_planned if planned else lib.fk_paged_decode_attn
    if split_weights:
        fn = functools.partial(lib.fk_paged_decode_attn_2p, int(planned))
    check(fn(
        _ptr(q), q.stride(0) if b else hq * d, _ptr(out), out.stride(0) if b else hq * d,
        _ptr(k_cache), _ptr(v_cache), nb, bs, k_cache.stride(0), int(kv_layout == "HND"),
        _ptr(context_lens), _ptr(block_tables), block_tables.stride(0) if b else 1,
        b, hq, hkv, d, float(softmax_scale), int(max_splits),
        _ptr(workspace), workspace.numel() * workspace.element_size(),
        _status_ptr(status, q), _stream()), "fk_paged_decode_attn")
    return out


def prefill_attn(q, k, v, cu_seqlens_q, cu_seqlens_k, max_seqlen_q, softmax_scale,
                 causal=True, block_table=None, kv_layout="NHD", out=None,
                 return_lse=False, status=None, split_weights=False):
    """Variable-length prefill attention on q [total_q, Hq, 128].  With split_weights
    `out` may keep fewer channels per head: [total_q, Hq, a multiple of 8].

    Without block_table, k / v are dense [total_k, Hkv, 128] (token-strided views
    allowed) and sequence i owns rows cu_seqlens_k[i]..cu_seqlens_k[i+1].  With
    block_table [num_seqs, cols] they are the paged pools (NHD
    [blocks, page, Hkv, 128] or HND [blocks, Hkv, page, 128]) and only the
    per-sequence key counts of cu_seqlens_k are used.  Causal masking is aligned
    to the END of each sequence's keys (a chunk of q_len queries after a cached
    prefix sees the prefix plus its own past).  split_weights: the fp32 weights enter
    P V as two bf16 parts instead of one.  Returns out, or (out, lse) with lse fp32
    [Hq, total_q]."""
    _need(q, BF16, "q")
    _need(k, BF16, "k")
    _need(v, BF16, "v")
    _need(cu_seqlens_q, torch.int32, "cu_seqlens_q")
    _need(cu_seqlens_k, torch.int32, "cu_seqlens_k")
    if q.dim() != 3 or q.stride(2) != 1 or q.stride(1) != q.shape[2]:
        raise _lib.FkError("q must be [total_q, Hq, D] with dense heads")
    total_q, hq, d = q.shape
    num_seqs = cu_seqlens_q.numel() - 1
    if cu_seqlens_k.numel() != num_seqs + 1:
        raise _lib.FkError("cu_seqlens_q and cu_seqlens_k must have the same length")
    if out is None:
        out = torch.empty((total_q, hq, d), dtype=BF16, device=q.device)
    elif out.stride(2) != 1 or out.stride(1) != out.shape[2] or \
            (out.shape[2] != d and not split_weights):
        raise _lib.FkError("out heads must be dense")
    lse = torch.empty((hq, total_q), dtype=torch.float32, device=q.device) if return_lse else None
    if block_table is None:
        if k.dim() != 3 or k.stride(2) != 1 or k.stride(1) != d or v.stride() != k.stride() \
                or v.shape != k.shape:
            raise _lib.FkError("dense k / v must be [total_k, Hkv, D] with dense heads")
        total_k, hkv = k.shape[0], k.shape[1]
        nb, bs, kv_stride, bt_stride = 0, 0, k.stride(0) if total_k else hkv * d, 0
    else:
        _need(block_table, torch.int32, "block_table")
        if block_table.stride(1) != 1:
            raise _lib.FkError("block_table rows must be dense")
        if kv_layout == "HND":
            nb, hkv, bs, d2 = k.shape
            dense = (bs * d2, d2, 1)
        else:
            nb, bs, hkv, d2 = k.shape
            dense = (hkv * d2, d2, 1)
        if d2 != d or v.shape != k.shape:
            raise _lib.FkError("cache shape mismatch")
        if k.stride()[1:] != dense or v.stride() != k.stride():
            raise _lib.FkError("caches must be dense within a block")
        total_k, kv_stride, bt_stride = 0, k.stride(0), block_table.stride(0)
    fn = lib.fk_prefill_attn_2p if split_weights else lib.fk_prefill_attn
    head = (out.shape[2],) if split_weights else ()
    check(fn(
        _ptr(q), q.stride(0) if total_q else hq * d, _ptr(out),
        out.stride(0) if total_q else hq * d, _ptr(lse), _ptr(k), _ptr(v), kv_stride, nb, bs,
        int(kv_layout == "HND"), _ptr(cu_seqlens_q), _ptr(cu_seqlens_k), _ptr(block_table),
        bt_stride, num_seqs, total_q, total_k, int(max_seqlen_q), hq, hkv, d, *head,
        float(softmax_scale), int(bool(causal)), _status_ptr(status, q), _stream()),
        "fk_prefill_attn")
    return (out, lse) if return_lse else out


def merge_attn_states(output, prefix_output, prefix_lse, suffix_output, suffix_lse,
                      output_lse=None, prefill_tokens_with_context=None) -> None:
    """output = log-sum-exp weighted mix of two partial attention results
    [T, H, D] bf16 with lse fp32 [H, T]; written in place (output_lse optional)."""
    for name, t in (("output", output), ("prefix_output", prefix_output),
                    ("suffix_output", suffix_output)):
        _need(t, BF16, name)
        if t.dim() != 3 or t.stride(2) != 1:
            raise _lib.FkError(f"{name} must be [T, H, D] with dense rows")
    for name, t in (("prefix_lse", prefix_lse), ("suffix_lse", suffix_lse)):
        _need(t, torch.float32, name)
        if not t.is_contiguous():
            raise _lib.FkError(f"{name} must be contiguous [H, T]")
    if output_lse is not None:
        _need(output_lse, torch.float32, "output_lse")
        if not output_lse.is_contiguous():
            raise _lib.FkError("output_lse must be contiguous [H, T]")
    t, h, d = output.shape
    if prefix_output.shape != output.shape or suffix_output.shape != output.shape:
        raise _lib.FkError("merge_attn_states: shape mismatch")
    check(lib.fk_merge_attn_states(
        _ptr(output), output.stride(0), output.stride(1), _ptr(output_lse),
        _ptr(prefix_output), prefix_output.stride(0), prefix_output.stride(1),
        _ptr(prefix_lse), _ptr(suffix_output), suffix_output.stride(0),
        suffix_output.stride(1), _ptr(suffix_lse), t, h, d,
        -1 if prefill_tokens_with_context is None else int(prefill_tokens_with_context),
        _stream()), "fk_merge_attn_states")


# --------------------------------------------------------------------------- norms
def rmsnorm(x, weight, eps, out=None):
    """out = bf16(x * rsqrt(mean(x^2)+eps) * w); x is [..., cols], last dim dense.
    2-D [T, cols] and 3-D [N, H, cols] (strided views allowed) are supported."""
    _need(x, BF16, "x")
    _need(weight, BF16, "weight")
    if x.stride(-1) != 1:
        raise _lib.FkError("x rows must be dense")
    cols = x.shape[-1]
    if out is None:
        out = torch.empty(x.shape, dtype=BF16, device=x.device)
    if x.dim() == 2:
        outer, inner = x.shape[0], 1
        xs = (x.stride(0) if outer else cols, 0)
        os_ = (out.stride(0) if outer else cols, 0)
    elif x.dim() == 3:
        outer, inner = x.shape[0], x.shape[1]
        xs = (x.stride(0), x.stride(1))
        os_ = (out.stride(0), out.stride(1))
    else:
        raise _lib.FkError("rmsnorm supports 2-D and 3-D inputs")
    check(lib.fk_rmsnorm(_ptr(x), xs[0], xs[1], inner, _ptr(out), os_[0], os_[1],
                         _ptr(weight), float(eps), outer, cols, _stream()), "fk_rmsnorm")
    return out


def fused_add_rmsnorm(x, residual, weight, eps) -> None:
    """In place: residual = bf16(x + residual); x = rmsnorm(residual) * w."""
    _need(x, BF16, "x")
    _need(residual, BF16, "residual")
    _need(weight, BF16, "weight")
    if x.dim() != 2 or residual.shape != x.shape or x.stride(1) != 1 or residual.stride(1) != 1:
        raise _lib.FkError("fused_add_rmsnorm needs matching 2-D row-dense tensors")
    rows, cols = x.shape
    check(lib.fk_fused_add_rmsnorm(_ptr(x), x.stride(0) if rows else cols, _ptr(residual),
                                   residual.stride(0) if rows else cols, _ptr(weight),
                                   float(eps), rows, cols, _stream()),
          "fk_fused_add_rmsnorm")


# ---------------------------------------------------------------------------- rope
def rope_neox(positions, query, key, head_dim, cos_sin_cache, status=None) -> None:
    """In-place NeoX rotation of query [T, Hq*D] and key [T, Hkv*D]."""
    _need(query, BF16, "query")
    _need(positions, torch.int64, "positions")
    t = query.shape[0]
    q2 = query.view(t, -1)
    hq = q2.shape[1] // head_dim
    if key is not None:
        _need(key, BF16, "key")
        k2 = key.view(t, -1)
        hkv = k2.shape[1] // head_dim
        ks = k2.stride(0) if t else k2.shape[1]
    else:
        k2, hkv, ks = None, 0, 0
    if cos_sin_cache.dtype not in (torch.float32, BF16):
        raise _lib.FkError("cos_sin_cache must be fp32 or bf16")
    check(lib.fk_rope_neox(_ptr(positions), _ptr(q2), q2.stride(0) if t else q2.shape[1], hq,
                           _ptr(k2), ks, hkv, head_dim, _ptr(cos_sin_cache),
                           int(cos_sin_cache.dtype == torch.float32),
                           cos_sin_cache.shape[0], t, _status_ptr(status, query),
                           _stream()),
          "fk_rope_neox")


def qkv_rope_store(qkv, num_q_heads, num_kv_heads, head_dim, positions, cos_sin_cache,
                   q_norm_weight, k_norm_weight, eps, k_cache, v_cache, slot_mapping,
                   status=None, kv_layout="NHD") -> None:
    """Split + [per-head q/k RMSNorm] + NeoX RoPE in place on the packed qkv rows,
    and store rotated k / raw v into the paged cache at slot_mapping."""
    _need(qkv, BF16, "qkv")
    _need(positions, torch.int64, "positions")
    if qkv.dim() != 2 or qkv.stride(1) != 1:
        raise _lib.FkError("qkv must be 2-D row-dense")
    t = qkv.shape[0]
    num_slots, page = 0, 0
    if k_cache is not None:
        page = k_cache.shape[2] if kv_layout == "HND" else k_cache.shape[1]
        _need(slot_mapping, torch.int32, "slot_mapping")
        if not (k_cache.is_contiguous() and v_cache.is_contiguous()):
            raise _lib.FkError("caches must be contiguous")
        num_slots = k_cache.numel() // (num_kv_heads * head_dim)
    check(lib.fk_qkv_rope_store(
        _ptr(qkv), qkv.stride(0) if t else qkv.shape[1], num_q_heads, num_kv_heads, head_dim,
        _ptr(positions), _ptr(cos_sin_cache), int(cos_sin_cache.dtype == torch.float32),
        cos_sin_cache.shape[0], _ptr(q_norm_weight), _ptr(k_norm_weight), float(eps),
        _ptr(k_cache), _ptr(v_cache), _ptr(slot_mapping), num_slots, page,
        int(kv_layout == "HND"), t, _status_ptr(status, qkv), _stream()), "fk_qkv_rope_store")


# ---------------------------------------------------------------------------- silu
def silu_and_mul(x, out=None):
    _need(x, BF16, "x")
    if x.dim() != 2 or x.stride(1) != 1:
        raise _lib.FkError("silu_and_mul needs a 2-D row-dense input")
    rows, d2 = x.shape
    d = d2 // 2
    if out is None:
        out = torch.empty((rows, d), dtype=BF16, device=x.device)
    check(lib.fk_silu_and_mul(_ptr(x), x.stride(0) if rows else d2, _ptr(out),
                              out.stride(0) if rows else d, rows, d, _stream()),
          "fk_silu_and_mul")
    return out


# ---------------------------------------------------------------------------- fill
def fill_u32(t: torch.Tensor, value: int = 0) -> None:
    """Fill a contiguous tensor (byte size a multiple of 4) with a 32-bit pattern."""
    nbytes = t.numel() * t.element_size()
    if not t.is_contiguous() or nbytes % 4:
        raise _lib.FkError("fill_u32 needs a contiguous tensor of whole 32-bit words")
    check(lib.fk_fill_u32(_ptr(t), nbytes // 4, value, _stream()), "fk_fill_u32")


def xor_u32(t: torch.Tensor, out: torch.Tensor | None = None) -> torch.Tensor:
    """XOR of all 32-bit words of a contiguous tensor (byte size a multiple of 16)
    into the one-element int32 tensor `out` (made and zeroed when not given): a
    checksum, and a pure read stream for bandwidth measurements."""
    nbytes = t.numel() * t.element_size()
    if not t.is_contiguous() or nbytes % 16:
        raise _lib.FkError("xor_u32 needs a contiguous tensor of whole 16-byte groups")
    if out is None:
        out = torch.zeros(1, dtype=torch.int32, device=t.device)
    check(lib.fk_xor_u32(_ptr(t), nbytes // 4, _ptr(out), _stream()), "fk_xor_u32")
    return out


# -------------------------------------------------------------------------- argmax
def argmax_rows(x, out_val=None, out_idx=None):
    """(max as fp32, lowest index of the max) per row of a bf16 or fp32 [rows, cols]
    matrix."""
    if x.dtype != torch.float32:
        _need(x, BF16, "x")
    if x.dim() != 2 or x.stride(1) != 1:
        raise _lib.FkError("argmax_rows needs a 2-D row-dense input")
    rows, cols = x.shape
    if out_val is None:
        out_val = torch.empty(rows, dtype=torch.float32, device=x.device)
    if out_idx is None:
        out_idx = torch.empty(rows, dtype=torch.int64, device=x.device)
    fn = lib.fk_argmax_f32 if x.dtype == torch.float32 else lib.fk_argmax_bf16
    check(fn(_ptr(x), x.stride(0) if rows else cols, rows, cols,
             _ptr(out_val), _ptr(out_idx), _stream()), "fk_argmax")
    return out_val, out_idx


# ---------------------------------------------------------------------------- gemm
def gemm_workspace_bytes(m, n, k) -> int:
    return int(lib.fk_gemm_bf16_workspace_bytes(m, n, k))


_GEMM_WS: dict = {}


def gemm_workspace(device) -> torch.Tensor:
    """Per-device stream-K workspace (flags + fp32 partial tiles), sized for the
    largest m, zero-initialised once.  The kernel leaves it zeroed, and GEMMs on
    one stream run one after the other, so a single buffer serves them all; a
    caller that runs GEMMs concurrently on several streams passes its own."""
    key = torch.device(device)
    if key.index is None and key.type == "cuda":
        key = torch.device("cuda", torch.cuda.current_device())
    ws = _GEMM_WS.get(key)
    if ws is None:
        ws = torch.zeros(gemm_workspace_bytes(256, 1, 64), dtype=torch.uint8, device=key)
        _GEMM_WS[key] = ws
    return ws


def gemm_bf16(x, w, bias=None, out=None, workspace=None, status=None):
    """y = x @ w.T (+ bias): x [m, k], w [n, k] contiguous, y [m, n] bf16."""
    _need(x, BF16, "x")
    _need(w, BF16, "w")
    if x.dim() != 2 or x.stride(1) != 1 or not w.is_contiguous():
        raise _lib.FkError("gemm_bf16 needs row-dense x and contiguous w")
    m, k = x.shape
    n = w.shape[0]
    if out is None:
        out = torch.empty((m, n), dtype=BF16, device=x.device)
    if workspace is None:
        workspace = gemm_workspace(x.device)
    # m <= 256: the weight-streaming decode kernel; more rows (prefill): the 256 x 256
    # tile kernel inside the same entry point
    check(lib.fk_gemm_bf16(_ptr(x), x.stride(0) if m else k, _ptr(w), _ptr(bias), _ptr(out),
                           out.stride(0) if m else n, m, n, k, _ptr(workspace),
                           workspace.numel() * workspace.element_size(),
                           _status_ptr(status, x), _stream()), "fk_gemm_bf16")
    return out


def gemm_bf16_push(x, w, bias, dst, nranks: int, call_counters: int, workspace=None,
                   status=None) -> None:
    """x @ w.T (+ bias) stored tile by tile into the receive areas `dst` (ctypes
    array of `nranks` device addresses) of all tensor-parallel ranks instead of a
    local y; `call_counters` = device address of this rank's per-row call counters."""
    _need(x, BF16, "x")
    _need(w, BF16, "w")
    if x.dim() != 2 or x.stride(1) != 1 or not w.is_contiguous():
        raise _lib.FkError("gemm_bf16_push needs row-dense x and contiguous w")
    m, k = x.shape
    n = w.shape[0]
    if workspace is None:
        workspace = gemm_workspace(x.device)
    check(lib.fk_gemm_bf16_push(_ptr(x), x.stride(0) if m else k, _ptr(w), _ptr(bias), m, n, k,
                                _ptr(workspace), workspace.numel() * workspace.element_size(),
                                dst, nranks, call_counters, _status_ptr(status, x), _stream()),
          "fk_gemm_bf16_push")


def gemm_silu_mul_fusable(m: int, n: int, k: int) -> bool:
    """True when silu_and_mul(x @ w.T) for x [m, k], w [n, k] runs as one launch."""
    return bool(lib.fk_gemm_bf16_silu_mul_fusable(m, n, k))


def gemm_silu_mul(x, w, bias=None, out=None, workspace=None, status=None):
    """silu_and_mul(x @ w.T (+ bias)) in one launch: w = [gate; up] rows, result
    [m, n / 2].  Raises for shapes without the single-launch form (see
    gemm_silu_mul_fusable)."""
    _need(x, BF16, "x")
    _need(w, BF16, "w")
    if x.dim() != 2 or x.stride(1) != 1 or not w.is_contiguous():
        raise _lib.FkError("gemm_silu_mul needs row-dense x and contiguous w")
    m, k = x.shape
    n = w.shape[0]
    if out is None:
        out = torch.empty((m, n // 2), dtype=BF16, device=x.device)
    if workspace is None:
        workspace = gemm_workspace(x.device)
    check(lib.fk_gemm_bf16_silu_mul(_ptr(x), x.stride(0) if m else k, _ptr(w), _ptr(bias),
                                    _ptr(out), out.stride(0) if m else n // 2, m, n, k,
                                    _ptr(workspace),
                                    workspace.numel() * workspace.element_size(),
                                    _status_ptr(status, x), _stream()), "fk_gemm_bf16_silu_mul")
    return out


def gemm_act_mul(x, w, act, bias=None, out=None, workspace=None, status=None):
    """act(x @ wg.T (+ bias)) * (x @ wu.T (+ bias)), w = [wg; wu] rows: one launch where
    the shape has one (see gemm_silu_mul_fusable), else the projection followed by
    act_and_mul."""
    m, k = x.shape
    half = w.shape[0] // 2
    if x.dtype == BF16 and gemm_silu_mul_fusable(m, 2 * half, k):
        _need(x, BF16, "x")
        _need(w, BF16, "w")
        if x.stride(1) != 1 or not w.is_contiguous():
            raise _lib.FkError("gemm_act_mul needs row-dense x and contiguous w")
        if out is None:
            out = torch.empty((m, half), dtype=BF16, device=x.device)
        if workspace is None:
            workspace = gemm_workspace(x.device)
        check(lib.fk_gemm_bf16_act_mul(
            _ptr(x), x.stride(0) if m else k, _ptr(w), _ptr(bias), _ptr(out),
            out.stride(0) if m else half, m, 2 * half, k, int(act), _ptr(workspace),
            workspace.numel() * workspace.element_size(), _status_ptr(status, x), _stream()),
            "fk_gemm_bf16_act_mul")
        return out
    return act_and_mul(gemm(x, w, bias=bias, workspace=workspace, status=status), act, out=out)


def gemm(x, w, bias=None, out=None, workspace=None, status=None):
    """x @ w.T (+ bias) in the type of its operands: bf16 (tensor cores, fp32
    accumulation) or true fp32."""
    if bias is not None:
        _need(bias, x.dtype, "bias")
        if bias.shape != (w.shape[0],) or not bias.is_contiguous():
            raise _lib.FkError("bias must have one entry per row of w")
    if x.dtype != torch.float32:
        return gemm_bf16(x, w, bias=bias, out=out, workspace=workspace, status=status)
    _need(x, torch.float32, "x")
    _need(w, torch.float32, "w")
    if x.dim() != 2 or x.stride(1) != 1 or not w.is_contiguous():
        raise _lib.FkError("gemm needs row-dense x and contiguous w")
    m, k = x.shape
    n = w.shape[0]
    if out is None:
        out = torch.empty((m, n), dtype=torch.float32, device=x.device)
    check(lib.fk_gemm_f32(_ptr(x), x.stride(0) if m else k, _ptr(w), _ptr(bias), _ptr(out),
                          out.stride(0) if m else n, m, n, k, _stream()), "fk_gemm_f32")
    return out


# ------------------------------------- fp32 residual stream, linear-attention mixers
def _is_f32(t: torch.Tensor, name: str) -> int:
    if not t.is_cuda:
        raise _lib.FkError(f"{name} must be a CUDA tensor (no CPU path exists)")
    if t.dtype not in (BF16, torch.float32):
        raise _lib.FkError(f"{name} must be bf16 or fp32, got {t.dtype}")
    return int(t.dtype == torch.float32)


def embed_f32(table, ids, out=None, status=None):
    """fp32 residual rows table[ids]; table [vocab, stride] bf16 or fp32."""
    f32 = _is_f32(table, "table")
    _need(ids, torch.int64, "ids")
    if not table.is_contiguous():
        raise _lib.FkError("table must be contiguous")
    n, stride = ids.shape[0], table.shape[1]
    if out is None:
        out = torch.empty((n, stride), dtype=torch.float32, device=table.device)
    check(lib.fk_embed_f32(_ptr(table), f32, table.shape[0], _ptr(ids), _ptr(out), n, stride,
                           _status_ptr(status, table), _stream()), "fk_embed_f32")
    return out


def norm_shift(x, gain, width, eps, dtype, y=None, y_gain=None, x_out=None, shift=None,
               state=None, slots=None, positions=None, cu_portions=None, out=None, status=None):
    """x' = x + rms(y) * y_gain; h = rms(x') * gain; token shift of h (see
    fk_norm_shift).  x fp32 [T, stride]; returns (x', out of `dtype`)."""
    _need(x, torch.float32, "x")
    if x.dim() != 2 or not x.is_contiguous():
        raise _lib.FkError("norm_shift needs a contiguous [T, stride] residual")
    rows, stride = x.shape
    if out is None:
        out = torch.empty((rows, stride), dtype=dtype, device=x.device)
    f32 = _is_f32(out, "out")
    if y is not None:
        _need(y, out.dtype, "y")
        if y.shape != x.shape or y.stride(1) != 1:
            raise _lib.FkError("norm_shift: y must be row-dense with the residual's shape")
        if x_out is None:
            x_out = torch.empty_like(x) if shift is not None else x
    n_port = 0
    if shift is not None:
        _need(state, torch.float32, "state")
        _need(slots, torch.int32, "slots")
        _need(positions, torch.int64, "positions")
        _need(cu_portions, torch.int32, "cu_portions")
        if state.dim() != 2 or state.shape[1] != stride or not state.is_contiguous():
            raise _lib.FkError("norm_shift: state must be a contiguous [slots, stride]")
        n_port = cu_portions.numel() - 1
    check(lib.fk_norm_shift(
        _ptr(x), _ptr(x_out), _ptr(y), y.stride(0) if y is not None and rows else stride,
        _ptr(y_gain), _ptr(gain), _ptr(shift), _ptr(out), f32, _ptr(state),
        state.shape[0] if state is not None else 0, _ptr(slots), _ptr(positions),
        _ptr(cu_portions), n_port, rows, stride, int(width), float(eps),
        _status_ptr(status, x), _stream()), "fk_norm_shift")
    return (x if x_out is None else x_out), out


def branch_combine(a, b, weight_a, weight_b, gain_out, x, width, eps, gain=None, out=None):
    """x += rms((rms(a) * weight_a + rms(b) * weight_b) / 2) * gain_out in place;
    returns rms(x) * gain in the type of a (None when gain is None)."""
    f32 = _is_f32(a, "a")
    _need(b, a.dtype, "b")
    _need(x, torch.float32, "x")
    rows, stride = x.shape
    if a.shape != x.shape or b.shape != x.shape or a.stride(1) != 1 or \
            (rows and b.stride() != a.stride()) or not x.is_contiguous():
        raise _lib.FkError("branch_combine needs row-dense operands of one shape")
    if gain is not None and out is None:
        out = torch.empty((rows, stride), dtype=a.dtype, device=x.device)
    check(lib.fk_branch_combine(
        _ptr(a), _ptr(b), a.stride(0) if rows else stride, _ptr(weight_a), _ptr(weight_b),
        _ptr(gain_out), _ptr(gain), _ptr(x), _ptr(out), f32, rows, stride, int(width),
        float(eps), _stream()), "fk_branch_combine")
    return out


def rope_rms_store(q, k, q_out, k_cache, v_cache, slots, positions, cos_sin, rot_dims,
                   num_q_heads, num_kv_heads, head_dim, eps, status=None) -> None:
    """Interleaved partial rotation + weight-less RMS norm of q and k heads; k (and k
    as projected, as the value) to the paged pool [blocks, page, Hkv, padded_dim].
    q / k are column ranges of the packed projection rows; q_out is
    [T, Hkv * padded_group, padded_dim]."""
    f32 = _is_f32(q, "q")
    for name, t in (("k", k), ("q_out", q_out), ("k_cache", k_cache), ("v_cache", v_cache)):
        _need(t, q.dtype, name)
    _need(slots, torch.int32, "slots")
    _need(positions, torch.int64, "positions")
    _need(cos_sin, torch.float32, "cos_sin")
    rows = q.shape[0]
    if q.stride(1) != 1 or k.stride(1) != 1 or (rows and q.stride(0) != k.stride(0)):
        raise _lib.FkError("q and k must be column ranges of the same rows")
    if not (q_out.is_contiguous() and k_cache.is_contiguous() and v_cache.is_contiguous()
            and cos_sin.is_contiguous()):
        raise _lib.FkError("q_out, caches and cos_sin must be contiguous")
    if q_out.shape[1] % num_kv_heads or k_cache.shape[2:] != (num_kv_heads, q_out.shape[2]) or \
            cos_sin.shape[1] != max(rot_dims, 1):
        raise _lib.FkError("rope_rms_store: shape mismatch")
    check(lib.fk_rope_rms_store(
        _ptr(q), _ptr(k), q.stride(0) if rows else 0, f32, _ptr(q_out), _ptr(k_cache),
        _ptr(v_cache), _ptr(slots), k_cache.shape[0] * k_cache.shape[1], _ptr(positions),
        _ptr(cos_sin), cos_sin.shape[0], rot_dims, num_q_heads, num_kv_heads, head_dim,
        q_out.shape[1] // num_kv_heads, q_out.shape[2], float(eps), rows,
        _status_ptr(status, q), _stream()), "fk_rope_rms_store")


def act_and_mul(x, act, out=None):
    """act(x[:, :d]) * x[:, d:], bf16 or fp32."""
    f32 = _is_f32(x, "x")
    if x.dim() != 2 or x.stride(1) != 1:
        raise _lib.FkError("act_and_mul needs a 2-D row-dense input")
    rows, d = x.shape[0], x.shape[1] // 2
    if out is None:
        out = torch.empty((rows, d), dtype=x.dtype, device=x.device)
    check(lib.fk_act_and_mul(_ptr(x), x.stride(0) if rows else 2 * d, _ptr(out),
                             out.stride(0) if rows else d, f32, rows, d, int(act), _stream()),
          "fk_act_and_mul")
    return out


def delta_padded_dim(dim: int) -> int:
    """Key channels per head in the delta rule's packed operands and state."""
    n = int(lib.fk_delta_padded_dim(int(dim)))
    if n <= 0:
        raise _lib.FkError(f"delta rule: head size {dim} unsupported")
    return n


def delta_prepare(r, k, v, a, y1, w2, w0, a_bias, heads, dim, decay_scale, unit_eps,
                  cu_portions=None, packed=None):
    """Operands of the delta rule (fp32, opaque): in blocks of 8 tokens of the portions
    when cu_portions is given, else token by token.  r, k, v, a [T, heads * dim] and
    y1 [T, rank] are column ranges of the same rows; w2 [heads * dim, padded rank]."""
    f32 = _is_f32(k, "k")
    rows, rank = y1.shape
    for name, t in (("r", r), ("v", v), ("a", a), ("y1", y1), ("w2", w2)):
        _need(t, k.dtype, name)
        if t is not w2 and (t.stride(1) != 1 or (rows and t.stride(0) != k.stride(0))):
            raise _lib.FkError(f"{name} must be a column range of the packed rows")
    _need(w0, torch.float32, "w0")
    _need(a_bias, torch.float32, "a_bias")
    if not w2.is_contiguous() or w2.shape[0] != heads * dim:
        raise _lib.FkError("w2 must be contiguous [heads * dim, padded rank]")
    n_port = 0
    if cu_portions is not None:
        _need(cu_portions, torch.int32, "cu_portions")
        n_port = cu_portions.numel() - 1
    delta_padded_dim(dim)
    if packed is None:
        n = int(lib.fk_delta_packed_floats(rows, n_port, heads, dim, int(n_port > 0)))
        packed = torch.empty(n, dtype=torch.float32, device=k.device)
    check(lib.fk_delta_prepare(
        _ptr(r), _ptr(k), _ptr(v), _ptr(a), _ptr(y1), k.stride(0) if rows else 0, f32, _ptr(w2),
        w2.shape[1], _ptr(w0), _ptr(a_bias), _ptr(packed), int(n_port > 0), _ptr(cu_portions),
        n_port, rows, heads, dim, rank, float(decay_scale), float(unit_eps), _stream()),
        "fk_delta_prepare")
    return packed


def delta_scan(packed, state, cu_portions, slots, positions, blocked, out=None, status=None):
    """The recurrence over prepared operands (`blocked`: prepared with cu_portions);
    state [slots, heads, dim, padded_dim] fp32 is read and replaced.  Returns
    o [T, heads * dim] fp32."""
    _need(packed, torch.float32, "packed")
    _need(state, torch.float32, "state")
    _need(cu_portions, torch.int32, "cu_portions")
    _need(slots, torch.int32, "slots")
    _need(positions, torch.int64, "positions")
    rows, heads, dim = positions.shape[0], state.shape[1], state.shape[2]
    n_port = cu_portions.numel() - 1
    if not packed.is_contiguous() or not state.is_contiguous() or \
            state.shape[3] != delta_padded_dim(dim) or packed.numel() < \
            int(lib.fk_delta_packed_floats(rows, n_port, heads, dim, int(bool(blocked)))):
        raise _lib.FkError("delta_scan: packed or state has the wrong shape")
    if out is None:
        out = torch.empty((rows, heads * dim), dtype=torch.float32, device=packed.device)
    check(lib.fk_delta_scan(
        _ptr(packed), int(bool(blocked)), _ptr(out), _ptr(state), state.shape[0],
        _ptr(cu_portions), n_port, _ptr(slots), _ptr(positions), rows, heads, dim,
        _status_ptr(status, packed), _stream()), "fk_delta_scan")
    return out


def head_norm_gate(o, gate, weight, heads, dim, eps, out):
    """out = rms(o per head) * weight * sigmoid(gate); columns of out beyond
    heads * dim are zeroed."""
    _need(o, torch.float32, "o")
    f32 = _is_f32(gate, "gate")
    _need(out, gate.dtype, "out")
    _need(weight, torch.float32, "weight")
    rows = o.shape[0]
    if not o.is_contiguous() or not out.is_contiguous() or gate.stride(1) != 1:
        raise _lib.FkError("head_norm_gate needs dense operands")
    check(lib.fk_head_norm_gate(_ptr(o), _ptr(gate), gate.stride(0) if rows else heads * dim,
                              _ptr(weight), _ptr(out), out.shape[1], f32, rows, heads, dim,
                              float(eps), _stream()), "fk_head_norm_gate")
    return out


def paged_attn_any(q, k_cache, v_cache, cu_seqlens_q, kv_lens, block_tables, softmax_scale,
                   out=None, status=None):
    """Causal attention over the NHD pool without shape restrictions (bf16 or fp32):
    the path for fp32 and for head sizes / GQA ratios the tensor-core kernels lack."""
    f32 = _is_f32(q, "q")
    _need(k_cache, q.dtype, "k_cache")
    _need(v_cache, q.dtype, "v_cache")
    for name, t in (("cu_seqlens_q", cu_seqlens_q), ("kv_lens", kv_lens),
                    ("block_tables", block_tables)):
        _need(t, torch.int32, name)
    rows, hq, d = q.shape
    nb, bs, hkv, d2 = k_cache.shape
    if d2 != d or v_cache.shape != k_cache.shape or not k_cache.is_contiguous() or \
            not v_cache.is_contiguous() or not q.is_contiguous() or block_tables.stride(1) != 1:
        raise _lib.FkError("paged_attn_any: shape or stride mismatch")
    if out is None:
        out = torch.empty((rows, hq, d), dtype=q.dtype, device=q.device)
    check(lib.fk_paged_attn_any(
        _ptr(q), hq * d, _ptr(out), out.stride(0) if rows else hq * d, _ptr(k_cache),
        _ptr(v_cache), f32, nb, bs, _ptr(cu_seqlens_q), _ptr(kv_lens), _ptr(block_tables),
        block_tables.stride(0), cu_seqlens_q.numel() - 1, rows, hq, hkv, d,
        float(softmax_scale), _status_ptr(status, q), _stream()), "fk_paged_attn_any")
    return out


# ----------------------------- parallel sublayers, latent attention, experts, matrix memory
def embed_pair_f32(table, ids, pairs=None, mul_prev=0, mul_cur=0, last_ids=None, slots=None,
                   positions=None, cu_portions=None, copy=None, status=None):
    """fp32 residual rows table[ids] (+ pairs[(previous token * mul_prev + token * mul_cur)
    mod buckets], the last row for a sequence's first token).  last_ids [slots] int64 keeps
    each sequence's last token; copy [T, stride]: the rows in the type of the tables too."""
    f32 = _is_f32(table, "table")
    _need(ids, torch.int64, "ids")
    n, stride = ids.shape[0], table.shape[1]
    if not table.is_contiguous():
        raise _lib.FkError("table must be contiguous")
    n_port = n_slots = 0
    if pairs is not None:
        _need(pairs, table.dtype, "pairs")
        _need(last_ids, torch.int64, "last_ids")
        _need(slots, torch.int32, "slots")
        _need(positions, torch.int64, "positions")
        _need(cu_portions, torch.int32, "cu_portions")
        if not pairs.is_contiguous() or pairs.shape[1] != stride:
            raise _lib.FkError("pairs must be contiguous rows of the table's width")
        n_port, n_slots = cu_portions.numel() - 1, last_ids.numel()
    if copy is not None:
        _need(copy, table.dtype, "copy")
        if copy.shape != (n, stride) or copy.stride(1) != 1:
            raise _lib.FkError("copy must be row-dense [T, stride]")
    x = torch.empty((n, stride), dtype=torch.float32, device=table.device)
    check(lib.fk_embed_pair_f32(
        _ptr(table), _ptr(pairs), f32, table.shape[0],
        pairs.shape[0] - 1 if pairs is not None else 0, int(mul_prev), int(mul_cur), _ptr(ids),
        _ptr(last_ids), n_slots, _ptr(slots), _ptr(positions), _ptr(cu_portions), n_port, _ptr(x),
        _ptr(copy), copy.stride(0) if copy is not None and n else stride, n, stride,
        _status_ptr(status, table), _stream()), "fk_embed_pair_f32")
    return x


def add_layernorm(x, width, eps, dtype, a=None, b=None, experts=None, norm1=None, norm2=None,
                  out1=None, out2=None, x_out=None, status=None):
    """x' = x + a + b + sum_j share[:, j] * rows[place[:, j]] (experts = (rows, place,
    share)), written to x_out (default: in place where something is added);
    norm1 / norm2 = (weight, bias) of layer norms of x', results of `dtype`.  Without norm1
    out1 (if given) gets x' itself.  Returns (x', out1, out2)."""
    _need(x, torch.float32, "x")
    if x.dim() != 2 or not x.is_contiguous():
        raise _lib.FkError("add_layernorm needs a contiguous [T, stride] residual")
    rows, stride = x.shape

    def like(t, name):
        if t is not None:
            _need(t, dtype, name)
            if t.shape[1] != stride or t.stride(1) != 1:
                raise _lib.FkError(f"{name} must be row-dense with the residual's width")
            return t.stride(0) if t.shape[0] else stride
        return stride
    if norm1 is not None and out1 is None:
        out1 = torch.empty((rows, stride), dtype=dtype, device=x.device)
    if norm2 is not None and out2 is None:
        out2 = torch.empty((rows, stride), dtype=dtype, device=x.device)
    f32 = int(dtype == torch.float32)
    if f32 == 0 and dtype != BF16:
        raise _lib.FkError("add_layernorm: bf16 or fp32")
    a_stride, b_stride = like(a, "a"), like(b, "b")
    e_rows, place, share = experts if experts is not None else (None, None, None)
    e_stride, top = like(e_rows, "experts"), 0
    if experts is not None:
        _need(place, torch.int32, "place")
        _need(share, torch.float32, "share")
        top = place.shape[1]
        if share.shape != place.shape or place.shape[0] != rows or \
                not place.is_contiguous() or not share.is_contiguous():
            raise _lib.FkError("place and share must be contiguous [T, top]")
    for name, nrm in (("norm1", norm1), ("norm2", norm2)):
        for t in nrm or ():
            _need(t, torch.float32, name)
            if t.numel() < stride or not t.is_contiguous():
                raise _lib.FkError(f"{name} must be padded to the residual's width")
    if x_out is None and (a is not None or b is not None or experts is not None):
        x_out = x
    w1, b1 = norm1 if norm1 is not None else (None, None)
    w2, b2 = norm2 if norm2 is not None else (None, None)
    check(lib.fk_add_layernorm(
        _ptr(x), _ptr(x_out), _ptr(a), a_stride, _ptr(b), b_stride, _ptr(e_rows), e_stride,
        e_rows.shape[0] if e_rows is not None else 0, _ptr(place), _ptr(share), top, _ptr(w1),
        _ptr(b1), _ptr(out1), like(out1, "out1"), _ptr(w2), _ptr(b2), _ptr(out2),
        like(out2, "out2"), f32, rows, stride, int(width), float(eps), _status_ptr(status, x),
        _stream()), "fk_add_layernorm")
    return (x if x_out is None else x_out), out1, out2


def softcap(x, cap):
    """cap * tanh(x / cap) in place."""
    f32 = _is_f32(x, "x")
    if x.dim() != 2 or x.stride(1) != 1:
        raise _lib.FkError("softcap needs a 2-D row-dense input")
    rows, cols = x.shape
    check(lib.fk_softcap(_ptr(x), x.stride(0) if rows else cols, f32, rows, cols, float(cap),
                         _stream()), "fk_softcap")
    return x


def group_gemm(x, w, out=None, bias=None, x_group=0, y_group=0, offsets=None, gather=None,
               rows=None, expect_rows=None, act=None, out_f32=False, status=None):
    """x w_g^T (+ bias) for w [groups, n (2 n with act), k] (or one [n, k]): column groups
    g take x[:, g * x_group:][:, :k] to out[:, g * y_group:][:, :n]; with offsets
    [groups + 1] group g takes the rows between its offsets (of x, or x[gather]).
    out_f32: fp32 result of bf16 operands.  See fk_group_gemm."""
    f32 = _is_f32(x, "x")
    _need(w, x.dtype, "w")
    if w.dim() == 2:
        w = w[None]
    if x.dim() != 2 or x.stride(1) != 1 or not w.is_contiguous():
        raise _lib.FkError("group_gemm needs row-dense x and contiguous w")
    groups, wn, k = w.shape
    n = wn if act is None else wn // 2
    if rows is None:
        rows = gather.shape[0] if gather is not None else x.shape[0]
    if expect_rows is None:
        expect_rows = rows if offsets is None else -(-rows // groups)
    y_type = torch.float32 if f32 or out_f32 else BF16
    if out is None:
        out = torch.empty((rows, n if offsets is not None or groups == 1
                           else (groups - 1) * y_group + n), dtype=y_type, device=x.device)
    _need(out, y_type, "out")
    for name, t in (("offsets", offsets), ("gather", gather)):
        if t is not None:
            _need(t, torch.int32, name)
    if offsets is not None and offsets.numel() != groups + 1:
        raise _lib.FkError("group_gemm: one offset per group and one more")
    if gather is not None and gather.numel() < rows:
        raise _lib.FkError("group_gemm: gather is shorter than the rows")
    if bias is not None:
        _need(bias, torch.float32, "bias")
        if bias.numel() < wn or not bias.is_contiguous():
            raise _lib.FkError("group_gemm: bias must have one entry per weight row")
    if out.dim() != 2 or out.shape[0] < rows or out.stride(1) != 1:
        raise _lib.FkError("group_gemm: out must be row-dense with a row per row")
    check(lib.fk_group_gemm(
        _ptr(x), x.stride(0) if x.shape[0] else x.shape[1], x_group, x.shape[0], _ptr(w),
        _ptr(bias), _ptr(out), out.stride(0) if rows else out.shape[1], y_group, f32,
        int(y_type == torch.float32), _ptr(offsets), _ptr(gather), rows, int(expect_rows),
        groups, n, k, -1 if act is None else int(act), _status_ptr(status, x), _stream()),
        "fk_group_gemm")
    return out


class Routing:
    """Which experts take which rows: chosen / share / place [T, top], source [T * top],
    offsets [experts + 1] (see fk_moe_route)."""

    def __init__(self, rows, experts, top, device):
        def ints(*shape):
            return torch.empty(shape, dtype=torch.int32, device=device)
        self.chosen, self.place = ints(rows, top), ints(rows, top)
        self.share = torch.empty((rows, top), dtype=torch.float32, device=device)
        self.source, self.offsets = ints(rows * top), ints(experts + 1)


def moe_route(z, top):
    """Routing from fp32 router logits [T, experts]."""
    _need(z, torch.float32, "z")
    if z.dim() != 2 or z.stride(1) != 1:
        raise _lib.FkError("moe_route needs 2-D row-dense logits")
    rows, experts = z.shape
    r = Routing(rows, experts, top, z.device)
    n = int(lib.fk_moe_route_counts(rows, experts, top))
    counts = torch.empty(n, dtype=torch.int32, device=z.device) if n else None
    check(lib.fk_moe_route(
        _ptr(z), z.stride(0) if rows else experts, _ptr(r.chosen), _ptr(r.share), _ptr(r.place),
        _ptr(r.source), _ptr(r.offsets), _ptr(counts), rows, experts, top, _stream()),
        "fk_moe_route")
    return r


def gather_rows(x, source, status=None):
    """x[source], rows of x a multiple of 16 bytes."""
    _need(source, torch.int32, "source")
    if not x.is_cuda or x.dim() != 2 or x.stride(1) != 1:
        raise _lib.FkError("gather_rows needs a row-dense CUDA matrix")
    out = torch.empty((source.numel(), x.shape[1]), dtype=x.dtype, device=x.device)
    size = x.element_size()
    check(lib.fk_gather_rows(_ptr(x), (x.stride(0) if x.shape[0] else x.shape[1]) * size,
                             x.shape[0], _ptr(source), _ptr(out), source.numel(),
                             x.shape[1] * size, _status_ptr(status, x), _stream()),
          "fk_gather_rows")
    return out


def latent_prepare(q, latent, q_pitch, weight, cos_sin, slots, positions, cache, q_out, q_rot_at,
                   copy, dim, rot, rank, eps, status=None) -> None:
    """Store the cached rows of latent attention and lay out its queries (see
    fk_latent_prepare).  q / latent are column ranges of the packed projection rows, cache
    [blocks, page, 1, pitch], q_out [T, heads, pitch]."""
    f32 = _is_f32(q, "q")
    for name, t in (("latent", latent), ("cache", cache), ("q_out", q_out)):
        _need(t, q.dtype, name)
    _need(weight, torch.float32, "weight")
    _need(cos_sin, torch.float32, "cos_sin")
    _need(slots, torch.int32, "slots")
    _need(positions, torch.int64, "positions")
    rows, heads = q_out.shape[:2]
    if q.stride(1) != 1 or latent.stride(1) != 1 or (rows and q.stride(0) != latent.stride(0)):
        raise _lib.FkError("q and latent must be column ranges of the same rows")
    if not (cache.is_contiguous() and q_out.is_contiguous() and cos_sin.is_contiguous()) or \
            q.shape[1] < (heads - 1) * q_pitch + dim + rot or latent.shape[1] < rank + rot or \
            cos_sin.shape[1] != max(rot, 1) or weight.numel() < rank:
        raise _lib.FkError("latent_prepare: shape mismatch")
    check(lib.fk_latent_prepare(
        _ptr(q), _ptr(latent), q.stride(0) if rows else 0, q_pitch, f32, _ptr(weight),
        _ptr(cos_sin), cos_sin.shape[0], _ptr(slots), _ptr(positions), _ptr(cache),
        cache.shape[0] * cache.shape[1], cache.shape[-1], _ptr(q_out), q_out.shape[2], q_rot_at,
        int(bool(copy)), rows, heads, dim, rot, rank, float(eps), _status_ptr(status, q),
        _stream()), "fk_latent_prepare")


def latent_gather(cache, block_tables, cu_seqlens_k, rows, status=None):
    """Cached rows [blocks, page, 1, pitch] of all sequences side by side: [rows, pitch]."""
    _need(block_tables, torch.int32, "block_tables")
    _need(cu_seqlens_k, torch.int32, "cu_seqlens_k")
    if not cache.is_cuda or not cache.is_contiguous() or block_tables.stride(1) != 1:
        raise _lib.FkError("latent_gather needs a contiguous CUDA pool and row-dense tables")
    pitch = cache.shape[-1]
    out = torch.empty((rows, pitch), dtype=cache.dtype, device=cache.device)
    check(lib.fk_latent_gather(
        _ptr(cache), pitch * cache.element_size(), cache.shape[0], cache.shape[1],
        _ptr(block_tables), block_tables.stride(0), _ptr(cu_seqlens_k),
        cu_seqlens_k.numel() - 1, _ptr(out), rows, _status_ptr(status, cache), _stream()),
        "fk_latent_gather")
    return out


def latent_attn_supported(rank: int, rot: int) -> bool:
    """True when fk_latent_attn takes rows of rank + rot channels."""
    return bool(lib.fk_latent_attn_supported(rank, rot))


def latent_attn(q, cache, cu_seqlens_q, kv_lens, block_tables, max_seqlen_q, max_keys, rank, rot,
                softmax_scale, out=None, status=None):
    """Absorbed latent attention, bf16: q [T, heads, pitch] over cached rows
    [blocks, page, 1, pitch] whose first `rank` channels are the values; out [T, heads,
    pitch].  max_keys bounds the keys of any sequence (it picks the number of key ranges)."""
    _need(q, BF16, "q")
    _need(cache, BF16, "cache")
    for name, t in (("cu_seqlens_q", cu_seqlens_q), ("kv_lens", kv_lens),
                    ("block_tables", block_tables)):
        _need(t, torch.int32, name)
    rows, heads, pitch = q.shape
    n_seq = cu_seqlens_q.numel() - 1
    if not q.is_contiguous() or not cache.is_contiguous() or block_tables.stride(1) != 1:
        raise _lib.FkError("latent_attn needs contiguous q and cache, row-dense tables")
    if out is None:
        out = torch.empty((rows, heads, (rank + 15) // 16 * 16), dtype=BF16, device=q.device)
    elif not out.is_contiguous():
        raise _lib.FkError("latent_attn: out must be contiguous")
    splits = int(lib.fk_latent_attn_splits(n_seq, int(max_seqlen_q), heads, rank,
                                           int(max_keys)))
    n = int(lib.fk_latent_attn_workspace_floats(rows, heads, rank, splits))
    ws = torch.empty(n, dtype=torch.float32, device=q.device) if n else None
    check(lib.fk_latent_attn(
        _ptr(q), pitch, _ptr(cache), cache.shape[0], cache.shape[1], cache.shape[-1], _ptr(out),
        out.shape[2], _ptr(cu_seqlens_q), _ptr(kv_lens), _ptr(block_tables),
        block_tables.stride(0), n_seq, rows, int(max_seqlen_q), heads, rank, rot,
        float(softmax_scale), splits, _ptr(ws), n, _status_ptr(status, q), _stream()),
        "fk_latent_attn")
    return out


def mlstm_state_shapes(num_slots, heads, dim, vdim):
    """Shapes of the two fp32 state tensors of a matrix memory."""
    return ((num_slots, heads, dim, int(lib.fk_mlstm_state_cols(vdim))),
            (num_slots, heads, int(lib.fk_mlstm_norm_cols(dim))))


def _mlstm_args(q, k, v, z, s_state, n_state, heads, dim, vdim):
    f32 = _is_f32(q, "q")
    for name, t in (("k", k), ("v", v)):
        _need(t, q.dtype, name)
    rows = q.shape[0]
    for name, t in (("q", q), ("k", k), ("v", v)):
        if t.stride(1) != 1 or (rows and t.stride(0) != q.stride(0)):
            raise _lib.FkError(f"{name} must be a column range of the packed rows")
    for name, t in (("z", z), ("s_state", s_state), ("n_state", n_state)):
        _need(t, torch.float32, name)
    if z.shape[1] < 2 * heads or z.stride(1) != 1 or not s_state.is_contiguous() or \
            not n_state.is_contiguous() or (s_state.shape, n_state.shape) != \
            mlstm_state_shapes(s_state.shape[0], heads, dim, vdim):
        raise _lib.FkError("matrix memory: gates or state have the wrong shape")
    return f32, rows


def mlstm_step(q, k, v, z, gate, weight, s_state, n_state, slots, positions, heads, dim, vdim,
               gate_cap, q_scale, eps, out, status=None):
    """One token per sequence: out = rms(o per head) * weight * sigmoid(gate)."""
    f32, rows = _mlstm_args(q, k, v, z, s_state, n_state, heads, dim, vdim)
    _need(out, q.dtype, "out")
    _need(gate, q.dtype, "gate")
    _need(weight, torch.float32, "weight")
    _need(slots, torch.int32, "slots")
    _need(positions, torch.int64, "positions")
    if out.stride(1) != 1 or gate.stride(1) != 1:
        raise _lib.FkError("mlstm_step needs row-dense operands")
    check(lib.fk_mlstm_step(
        _ptr(q), _ptr(k), _ptr(v), q.stride(0) if rows else 0, f32, _ptr(z),
        z.stride(0) if rows else 2 * heads, _ptr(gate), gate.stride(0) if rows else heads * vdim,
        _ptr(weight), _ptr(s_state), _ptr(n_state), s_state.shape[0], _ptr(slots),
        _ptr(positions), _ptr(out), out.stride(0) if rows else out.shape[1], rows, heads, dim,
        vdim, float(gate_cap), float(q_scale), float(eps), _status_ptr(status, q), _stream()),
        "fk_mlstm_step")
    return out


def mlstm_portions(q, k, v, z, s_state, n_state, cu_portions, slots, positions, heads, dim, vdim,
                   gate_cap, q_scale, longest, chunked=True, status=None):
    """The memory over portions; o [T, heads * vdim] fp32 ahead of norm and gate.  bf16
    goes 128 tokens at a time unless chunked is False."""
    f32, rows = _mlstm_args(q, k, v, z, s_state, n_state, heads, dim, vdim)
    _need(cu_portions, torch.int32, "cu_portions")
    _need(slots, torch.int32, "slots")
    _need(positions, torch.int64, "positions")
    n_port = cu_portions.numel() - 1
    o = torch.empty((rows, heads * vdim), dtype=torch.float32, device=q.device)
    ws, n = None, 0
    if chunked and not f32:
        n = int(lib.fk_mlstm_workspace_floats(rows, n_port, heads, dim, vdim))
        ws = torch.empty(n, dtype=torch.float32, device=q.device)
    check(lib.fk_mlstm_portions(
        _ptr(q), _ptr(k), _ptr(v), q.stride(0) if rows else 0, f32, _ptr(z),
        z.stride(0) if rows else 2 * heads, _ptr(s_state), _ptr(n_state), s_state.shape[0],
        _ptr(cu_portions), n_port, _ptr(slots), _ptr(positions), _ptr(o), rows, heads, dim, vdim,
        float(gate_cap), float(q_scale), _ptr(ws), n, int(longest), _status_ptr(status, q),
        _stream()), "fk_mlstm_portions")
    return o


# -------------------------------------------------------------------- decode block
class BlockProgram:
    """Builder for one fk_decode_block launch: the projections, residual-add +
    RMSNorms and the split + RoPE + KV store a decoder layer runs between two
    attention calls, executed by one persistent kernel.  Phases run in the order
    they are added; every tensor is bf16, row-dense, with m rows."""

    def __init__(self, m: int, device):
        self.m, self.device = int(m), torch.device(device)
        self.phases: list = []
        self._keep: list = []          # tensors referenced by raw pointers

    def _phase(self, kind):
        ph = _lib.BlockPhase()
        ph.kind = kind
        self.phases.append(ph)
        return ph

    def _gemm(self, kind, x, w, bias, out):
        _need(x, BF16, "x")
        _need(w, BF16, "w")
        if x.dim() != 2 or x.shape[0] != self.m or x.stride(1) != 1 or not w.is_contiguous():
            raise _lib.FkError("block projection needs row-dense x [m, k] and contiguous w")
        n, k = w.shape
        cols = n // 2 if kind == _lib.PHASE_GEMM_SILU_MUL else n
        if out is None:
            out = torch.empty((self.m, cols), dtype=BF16, device=x.device)
        ph = self._phase(kind)
        ph.x, ph.x_stride = x.data_ptr(), x.stride(0)
        ph.w, ph.bias = w.data_ptr(), _ptr(bias)
        ph.y, ph.y_stride = out.data_ptr(), out.stride(0)
        ph.n, ph.k = n, k
        self._keep += [x, w, bias, out]
        return out

    def gemm(self, x, w, bias=None, out=None):
        """out = x @ w.T (+ bias)"""
        return self._gemm(_lib.PHASE_GEMM, x, w, bias, out)

    def gemm_silu_mul(self, x, w, bias=None, out=None):
        """out = silu_and_mul(x @ w.T (+ bias)), w = [gate; up]"""
        if w.shape[0] % 128:
            raise _lib.FkError("gate/up projection rows must be a multiple of 128")
        return self._gemm(_lib.PHASE_GEMM_SILU_MUL, x, w, bias, out)

    def add_rmsnorm(self, x, residual, weight, eps, out=None):
        """residual += x (x None: nothing added); out = rmsnorm(residual) * weight"""
        _need(residual, BF16, "residual")
        _need(weight, BF16, "weight")
        if residual.dim() != 2 or residual.shape[0] != self.m or residual.stride(1) != 1:
            raise _lib.FkError("block norm needs a row-dense residual [m, cols]")
        if out is None:
            out = torch.empty_like(residual)
        ph = self._phase(_lib.PHASE_ADD_RMSNORM)
        if x is not None:
            _need(x, BF16, "x")
            if x.shape != residual.shape or x.stride(1) != 1:
                raise _lib.FkError("block norm: x and residual must have the same shape")
            ph.x, ph.x_stride = x.data_ptr(), x.stride(0)
        ph.residual, ph.residual_stride = residual.data_ptr(), residual.stride(0)
        ph.norm_weight, ph.eps = weight.data_ptr(), float(eps)
        ph.y, ph.y_stride = out.data_ptr(), out.stride(0)
        ph.n = residual.shape[1]
        self._keep += [x, residual, weight, out]
        return out

    def qkv_rope_store(self, qkv, num_q_heads, num_kv_heads, head_dim, positions,
                       cos_sin_cache, q_norm_weight, k_norm_weight, eps, k_cache, v_cache,
                       slot_mapping, kv_layout="NHD"):
        """ops.qkv_rope_store on the packed qkv rows (bf16 cos/sin cache)."""
        _need(qkv, BF16, "qkv")
        _need(positions, torch.int64, "positions")
        _need(cos_sin_cache, BF16, "cos_sin_cache")
        if qkv.dim() != 2 or qkv.shape[0] != self.m or qkv.stride(1) != 1:
            raise _lib.FkError("qkv must be row-dense [m, (Hq + 2 Hkv) * D]")
        ph = self._phase(_lib.PHASE_QKV_ROPE_STORE)
        ph.x, ph.x_stride = qkv.data_ptr(), qkv.stride(0)
        ph.num_q_heads, ph.num_kv_heads, ph.head_dim = num_q_heads, num_kv_heads, head_dim
        ph.positions = positions.data_ptr()
        ph.cos_sin_cache, ph.cache_is_fp32 = cos_sin_cache.data_ptr(), 0
        ph.max_position = cos_sin_cache.shape[0]
        ph.q_norm_weight, ph.k_norm_weight = _ptr(q_norm_weight), _ptr(k_norm_weight)
        ph.eps = float(eps)
        if k_cache is not None:
            _need(slot_mapping, torch.int32, "slot_mapping")
            if not (k_cache.is_contiguous() and v_cache.is_contiguous()):
                raise _lib.FkError("caches must be contiguous")
            ph.k_cache, ph.v_cache = k_cache.data_ptr(), v_cache.data_ptr()
            ph.slot_mapping = slot_mapping.data_ptr()
            ph.num_slots = k_cache.numel() // (num_kv_heads * head_dim)
            ph.block_size = k_cache.shape[2] if kv_layout == "HND" else k_cache.shape[1]
            ph.kv_layout = int(kv_layout == "HND")
        self._keep += [qkv, positions, cos_sin_cache, q_norm_weight, k_norm_weight, k_cache,
                       v_cache, slot_mapping]

    def launch(self, workspace=None, status=None) -> None:
        if not self.phases:
            return
        if workspace is None:
            workspace = gemm_workspace(self.device)
        arr = (_lib.BlockPhase * len(self.phases))(*self.phases)
        st = status if status is not None else default_status(self.device)
        check(lib.fk_decode_block(arr, len(self.phases), self.m, _ptr(workspace),
                                  workspace.numel() * workspace.element_size(), st.data_ptr(),
                                  _stream()), "fk_decode_block")


def decode_block_max_rows() -> int:
    return 128
