"""Sequence mixers on packed projection rows.

A mixer names the row blocks it wants from the projection that all mixers of a layer
share (`sections`), reads its columns of the projected rows, and leaves its output
(before the output projection) in a buffer whose columns match its packed output
weight.  State lives in per-pass pools that the model allocates: a layer that runs
several times in a row has one per pass.
"""
from __future__ import annotations

import math

import torch

from fastkernels_b200 import ops
from fastkernels_b200.infra.context import get_context


def round_up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


def rope_table(max_positions: int, rot_dims: int, base: float, device) -> torch.Tensor:
    """[max_positions, rot_dims] fp32 = cos | sin of p * base^(-2 i / rot_dims), the
    angles taken in 64-bit."""
    if rot_dims == 0:
        return torch.zeros((max_positions, 1), dtype=torch.float32, device=device)
    f = base ** (-torch.arange(0, rot_dims, 2, dtype=torch.float64, device=device) / rot_dims)
    a = torch.arange(max_positions, dtype=torch.float64, device=device)[:, None] * f
    return torch.cat([a.cos(), a.sin()], dim=1).float().contiguous()


class RotaryAttention:
    """Softmax attention whose values are the projected keys, with interleaved partial
    rotation and a weight-less RMS norm of q and k, over the paged pool of one span.

    bf16 with head sizes up to 128 runs on the tensor-core kernels, heads padded to
    128 channels and query groups to a power of two (zeros), the fp32 softmax weights in
    two bf16 parts; fp32 and everything else
    on fk_paged_attn_any.  The output weight is packed with the same padding."""

    def __init__(self, heads, kv_heads, dim, scale, rot_dims, rot_base, span, eps, dtype):
        if heads % kv_heads:
            raise ValueError("query heads must be a multiple of key/value heads")
        self.heads, self.kv_heads, self.dim = heads, kv_heads, dim
        self.scale, self.eps = scale, eps
        self.rot_dims, self.rot_base = rot_dims, rot_base
        self.span, self.dtype = span, dtype
        g = heads // kv_heads
        self.tensor_cores = dtype == torch.bfloat16 and dim <= 128 and g <= 16
        self.group = 1 << (g - 1).bit_length() if self.tensor_cores else g
        self.padded_dim = 128 if self.tensor_cores else round_up(dim, 4)
        self.sections = {"q": heads * dim, "k": kv_heads * dim}
        self.out_columns = round_up(kv_heads * self.group * self.padded_dim, 64)
        self.k_caches, self.v_caches = [], []
        self.cos_sin = self.plan = self.workspace = self.status = None
        self.max_splits = 1

    def pack_output(self, w: torch.Tensor) -> torch.Tensor:
        """[out, heads * dim] -> [out, out_columns] with the padding of the heads."""
        n = w.shape[0]
        full = torch.zeros((n, self.kv_heads, self.group, self.padded_dim), dtype=w.dtype,
                           device=w.device)
        full[:, :, :self.heads // self.kv_heads, :self.dim] = \
            w.view(n, self.kv_heads, -1, self.dim)
        out = torch.zeros((n, self.out_columns), dtype=w.dtype, device=w.device)
        out[:, :self.kv_heads * self.group * self.padded_dim] = full.view(n, -1)
        return out

    def allocate(self, passes, num_blocks, block_size, device):
        shape = (num_blocks, block_size, self.kv_heads, self.padded_dim)
        pools = [torch.zeros((2, *shape), dtype=self.dtype, device=device)
                 for _ in range(passes)]
        self.k_caches = [p[0] for p in pools]
        self.v_caches = [p[1] for p in pools]
        return pools

    @property
    def plan_key(self):
        return self.span, self.kv_heads * self.group, self.kv_heads

    def forward(self, cols, positions, run):
        """cols: {section: its columns of the packed rows}."""
        span = get_context().spans[self.span]
        t = positions.shape[0]
        width = self.kv_heads * self.group * self.padded_dim
        q = torch.empty((t, self.kv_heads * self.group, self.padded_dim), dtype=self.dtype,
                        device=positions.device)
        kc, vc = self.k_caches[run], self.v_caches[run]
        ops.rope_rms_store(cols["q"], cols["k"], q, kc, vc, span.slot_mapping, positions,
                           self.cos_sin, self.rot_dims, self.heads, self.kv_heads, self.dim,
                           self.eps, status=self.status)
        alloc = torch.empty if width == self.out_columns else torch.zeros
        out = alloc((t, self.out_columns), dtype=self.dtype, device=positions.device)
        heads = out[:, :width].unflatten(1, (self.kv_heads * self.group, self.padded_dim))
        if not self.tensor_cores:
            ops.paged_attn_any(q, kc, vc, span.cu_seqlens_q, span.kv_lens, span.block_tables,
                               self.scale, out=heads, status=self.status)
        elif get_context().is_prefill:
            ops.prefill_attn(q, kc, vc, span.cu_seqlens_q, span.cu_seqlens_k, span.max_seqlen_q,
                             self.scale, block_table=span.block_tables, out=heads,
                             status=self.status, split_weights=True)
        else:
            ops.paged_decode_attn(q, kc, vc, span.kv_lens, span.block_tables, self.scale,
                                  self.workspace, self.max_splits, out=heads,
                                  status=self.status, planned=self.plan, split_weights=True)
        return out


class GeneralizedDelta:
    """Linear attention with a per-channel decay and a delta-rule removal term (see
    fk_delta_scan), heads x dim keys and values, and a gated per-head RMS norm."""

    DECAY_SCALE = math.exp(-0.5)
    UNIT_EPS = 1e-6

    def __init__(self, heads, dim, rank, eps, dtype):
        self.heads, self.dim, self.rank, self.eps, self.dtype = heads, dim, rank, eps, dtype
        hd = heads * dim
        self.sections = {"r": hd, "k": hd, "v": hd, "a": hd, "g": hd, "w1": rank}
        self.out_columns = round_up(hd, 64)
        self.w0 = self.w2 = self.a_bias = self.norm = self.status = None
        self.states = []

    def pack_output(self, w):
        out = torch.zeros((w.shape[0], self.out_columns), dtype=w.dtype, device=w.device)
        out[:, :w.shape[1]] = w
        return out

    def allocate(self, passes, num_slots, device):
        self.states = [torch.zeros((num_slots, self.heads, self.dim,
                                    ops.delta_padded_dim(self.dim)), dtype=torch.float32,
                                   device=device) for _ in range(passes)]

    def forward(self, cols, positions, run):
        ctx = get_context()
        packed = ops.delta_prepare(cols["r"], cols["k"], cols["v"], cols["a"], cols["w1"],
                                   self.w2, self.w0, self.a_bias, self.heads, self.dim,
                                   self.DECAY_SCALE, self.UNIT_EPS,
                                   cu_portions=ctx.cu_portions if ctx.is_prefill else None)
        o = ops.delta_scan(packed, self.states[run], ctx.cu_portions, ctx.state_slots, positions,
                           ctx.is_prefill, status=self.status)
        out = torch.empty((positions.shape[0], self.out_columns), dtype=self.dtype,
                          device=positions.device)
        return ops.delta_output(o, cols["g"], self.norm, self.heads, self.dim, self.eps, out)
