"""Sequence mixers on packed projection rows.

A mixer names the row blocks it wants from the projection that all mixers of a layer
share (`sections`), reads its columns of the projected rows, and leaves its output
(before the output projection) in a buffer whose columns match its packed output
weight.  State lives in per-pass pools that the model allocates: a layer that runs
several times in a row has one per pass.
"""
from __future__ import annotations

import math
from dataclasses import dataclass

import torch

from fastkernels_b200 import ops
from fastkernels_b200.infra.context import get_context


def round_up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


@dataclass(frozen=True)
class Yarn:
    """YaRN scaling of rotary frequencies: pairs that turn fewer than `slow` times over
    `original` positions are slowed by `factor`, those that turn more than `fast` times stay,
    the ones between are blended; cos and sin grow by 0.1 ln(factor) + 1."""
    factor: float
    original: float
    fast: float
    slow: float

    def apply(self, f: torch.Tensor, rot_dims: int, base: float) -> torch.Tensor:
        def pair(turns):
            return rot_dims * math.log(self.original / (2 * math.pi * turns)) \
                / (2 * math.log(base))
        lo = max(math.floor(pair(self.fast)), 0)
        hi = min(math.ceil(pair(self.slow)), rot_dims - 1)
        i = torch.arange(f.numel(), dtype=torch.float64, device=f.device)
        ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        return f / self.factor * ramp + f * (1.0 - ramp)

    @property
    def magnitude(self) -> float:
        return 0.1 * math.log(self.factor) + 1.0


def rope_table(max_positions: int, rot_dims: int, base: float, device,
               scaling: Yarn | None = None) -> torch.Tensor:
    """[max_positions, rot_dims] fp32 = cos | sin of p * base^(-2 i / rot_dims), the
    angles taken in 64-bit; `scaling` changes the frequencies and the magnitude."""
    if rot_dims == 0:
        return torch.zeros((max_positions, 1), dtype=torch.float32, device=device)
    f = base ** (-torch.arange(0, rot_dims, 2, dtype=torch.float64, device=device) / rot_dims)
    if scaling is not None:
        f = scaling.apply(f, rot_dims, base)
    a = torch.arange(max_positions, dtype=torch.float64, device=device)[:, None] * f
    size = 1.0 if scaling is None else scaling.magnitude
    return (torch.cat([a.cos(), a.sin()], dim=1) * size).float().contiguous()


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
        return ops.head_norm_gate(o, cols["g"], self.norm, self.heads, self.dim, self.eps, out)


class LatentAttention:
    """Softmax attention over one cached row per token: a normed latent of `rank` channels,
    from which every head makes its unrotated key and its value, and a rotated key of `rot`
    channels that all heads share.

    Two forms of the same sums.  Absorbed: a head's key projection is applied to its query and
    its value projection to its output, so attention runs on the cached rows themselves
    (decoding, short portions, fp32, heads above 128 channels).  Expanded: keys and values of
    all heads are made from the cached rows by one product (the rotated part passes through
    an identity block) and attention runs on the tcgen05 prefill kernel."""

    # expanded attention makes keys and values of every visible token: worth it for portions
    # that are not much shorter than what they see
    EXPAND_RATIO = 8

    def __init__(self, heads, dim, rot, vdim, rank, scale, rot_base, rot_scaling, span, eps,
                 dtype):
        self.heads, self.dim, self.rot, self.vdim, self.rank = heads, dim, rot, vdim, rank
        self.scale, self.rot_base, self.rot_scaling = scale, rot_base, rot_scaling
        self.span, self.eps, self.dtype = span, eps, dtype
        self.q_pitch = round_up(dim + rot, 8)
        self.row = round_up(rank + rot, 64)              # elements of a cached row
        self.v_pitch = round_up(vdim, 8)
        self.out_columns = round_up(heads * self.v_pitch, 64)
        self.sections = {"q": heads * self.q_pitch, "dkv": rank + rot}
        self.tensor_cores = dtype == torch.bfloat16 and ops.latent_attn_supported(rank, rot)
        self.expandable = dtype == torch.bfloat16 and dim + rot <= 128 and vdim <= 128
        self.caches = []
        self.cos_sin = self.status = None

    def load(self, w, prefix) -> dict:
        """Packs the weights; returns the rows of the shared projection by section."""
        h, d, r, k = self.heads, self.dim, self.rot, self.rank
        q = w.zeros(h, self.q_pitch, w.width)
        q[:, :d + r] = w.matrix(prefix + "q").view(h, d + r, -1)
        uk = w.matrix(prefix + "uk").view(h, d, k)
        uv = w.matrix(prefix + "uv").view(h, self.vdim, k)
        self.norm = w.vector(prefix + "dkv.norm")
        # absorbed: query [rank, dim] and value [vdim, rank] per head
        self.w_key = w.zeros(h, k, round_up(d, 16))
        self.w_key[:, :, :d] = uk.transpose(1, 2)
        self.w_value = w.zeros(h, self.v_pitch, round_up(k, 16))
        self.w_value[:, :self.vdim, :k] = uv
        if self.expandable:
            self.w_expand = w.zeros(2, h, 128, self.row)
            self.w_expand[0, :, :d, :k] = uk
            self.w_expand[0, :, d:d + r, k:k + r] = torch.eye(r, dtype=w.dtype, device=w.device)
            self.w_expand[1, :, :self.vdim, :k] = uv
            self.w_expand = self.w_expand.view(2 * h * 128, self.row)
        return {"q": q.view(h * self.q_pitch, -1), "dkv": w.matrix(prefix + "dkv")}

    def pack_output(self, w: torch.Tensor) -> torch.Tensor:
        n = w.shape[0]
        full = torch.zeros((n, self.heads, self.v_pitch), dtype=w.dtype, device=w.device)
        full[:, :, :self.vdim] = w.view(n, self.heads, self.vdim)
        out = torch.zeros((n, self.out_columns), dtype=w.dtype, device=w.device)
        out[:, :self.heads * self.v_pitch] = full.view(n, -1)
        return out

    def allocate(self, passes, num_blocks, block_size, device):
        self.caches = [torch.zeros((num_blocks, block_size, 1, self.row), dtype=self.dtype,
                                   device=device) for _ in range(passes)]
        return self.caches

    def forward(self, h, cols, positions, run):
        """h: input rows (not read here); cols: {section: its columns of the packed rows}."""
        ctx = get_context()
        span = ctx.spans[self.span]
        t, cache = positions.shape[0], self.caches[run]
        width = self.heads * self.v_pitch
        alloc = torch.empty if width == self.out_columns else torch.zeros
        out = alloc((t, self.out_columns), dtype=self.dtype, device=positions.device)
        expand = self.expandable and ctx.is_prefill and \
            span.total_k <= self.EXPAND_RATIO * t
        q = torch.empty((t, self.heads, 128 if expand else self.row), dtype=self.dtype,
                        device=positions.device)
        ops.latent_prepare(cols["q"], cols["dkv"], self.q_pitch, self.norm, self.cos_sin,
                           span.slot_mapping, positions, cache, q,
                           self.dim if expand else self.rank, expand, self.dim, self.rot,
                           self.rank, self.eps, status=self.status)
        if expand:
            rows = ops.latent_gather(cache, span.block_tables, span.cu_seqlens_k, span.total_k,
                                     status=self.status)
            kv = ops.group_gemm(rows, self.w_expand, status=self.status)
            kv = kv.view(span.total_k, 2, self.heads, 128)
            ops.prefill_attn(q, kv[:, 0], kv[:, 1], span.cu_seqlens_q, span.cu_seqlens_k,
                             span.max_seqlen_q, self.scale,
                             out=out[:, :width].unflatten(1, (self.heads, self.v_pitch)),
                             status=self.status, split_weights=True)
            return out
        ops.group_gemm(cols["q"], self.w_key, out=q.view(t, -1), x_group=self.q_pitch,
                       y_group=self.row, status=self.status)
        if self.tensor_cores:
            keys = span.max_seqlen_k if ctx.is_prefill else \
                span.block_tables.shape[1] * cache.shape[1]
            o = ops.latent_attn(q, cache, span.cu_seqlens_q, span.kv_lens, span.block_tables,
                                span.max_seqlen_q, keys, self.rank, self.rot, self.scale,
                                status=self.status)
        else:
            o = ops.paged_attn_any(q, cache, cache, span.cu_seqlens_q, span.kv_lens,
                                   span.block_tables, self.scale, status=self.status)
        ops.group_gemm(o.view(t, -1), self.w_value, out=out, x_group=o.shape[2],
                       y_group=self.v_pitch, status=self.status)
        return out


class MatrixMemory:
    """Matrix memory with exponential gating (see fk_mlstm_step): heads of dim x vdim, a
    normalizer and a running maximum per head, per-head RMS norm and output gate."""

    def __init__(self, heads, dim, vdim, gate_cap, eps, dtype):
        self.heads, self.dim, self.vdim, self.gate_cap = heads, dim, vdim, gate_cap
        self.eps, self.dtype = eps, dtype
        self.sections = {"q": heads * dim, "k": heads * dim, "v": heads * vdim,
                         "g": heads * vdim}
        self.out_columns = round_up(heads * vdim, 64)
        self.status = None
        self.states = []

    def load(self, w, prefix) -> dict:
        # the gates' pre-activations stay fp32, so they are a product of their own
        self.w_gates = w.padded(torch.cat([w.matrix(prefix + n) for n in "if"]),
                                2 * self.heads, w.stride)
        self.b_gates = torch.cat([w.vector(f"{prefix}{n}.b") for n in "if"])
        self.norm = w.vector(prefix + "norm")
        return {n: w.matrix(prefix + n) for n in "qkvg"}

    def pack_output(self, w):
        out = torch.zeros((w.shape[0], self.out_columns), dtype=w.dtype, device=w.device)
        out[:, :w.shape[1]] = w
        return out

    def allocate(self, passes, num_slots, device):
        shapes = ops.mlstm_state_shapes(num_slots, self.heads, self.dim, self.vdim)
        self.states = [tuple(torch.zeros(s, dtype=torch.float32, device=device) for s in shapes)
                       for _ in range(passes)]

    def forward(self, h, cols, positions, run):
        ctx = get_context()
        z = ops.group_gemm(h, self.w_gates, bias=self.b_gates, out_f32=True, status=self.status)
        out = torch.empty((positions.shape[0], self.out_columns), dtype=self.dtype,
                          device=positions.device)
        scale = self.dim ** -0.5
        if not ctx.is_prefill:
            return ops.mlstm_step(cols["q"], cols["k"], cols["v"], z, cols["g"], self.norm,
                                  *self.states[run], ctx.state_slots, positions, self.heads,
                                  self.dim, self.vdim, self.gate_cap, scale, self.eps, out,
                                  status=self.status)
        o = ops.mlstm_portions(cols["q"], cols["k"], cols["v"], z, *self.states[run],
                               ctx.cu_portions, ctx.state_slots, positions, self.heads, self.dim,
                               self.vdim, self.gate_cap, scale, ctx.longest_portion,
                               status=self.status)
        return ops.head_norm_gate(o, cols["g"], self.norm, self.heads, self.vdim, self.eps, out)
