"""Feed-forward sublayers on padded rows.

`forward(h)` returns (dense, experts): rows to add to the residual, and the rows of a
mixture as ops.add_layernorm takes them (rows, place, share), or None.
"""
from __future__ import annotations

import torch

from fastkernels_b200 import _lib, ops

from .mixers import round_up


class GatedFeedForward:
    """down(act(gate h) * (up h)), with or without biases."""

    # rows from which the many-row grouped product (activation in its epilogue) takes over
    # from the projection with a kernel for the activation behind it
    MANY_ROWS = 256

    def __init__(self, ff: int, bias: bool, act: int = _lib.ACT_SILU):
        self.ff, self.bias, self.act = ff, bias, act
        self.status = None

    @staticmethod
    def tensor_shapes(prefix, width, ff, bias) -> dict:
        s = {prefix + "gate": (ff, width), prefix + "up": (ff, width), prefix + "down": (width, ff)}
        if bias:
            s.update({prefix + "gate.b": (ff,), prefix + "up.b": (ff,),
                      prefix + "down.b": (width,)})
        return s

    def load(self, w, prefix) -> None:
        ff = round_up(self.ff, 64)
        self.w_gate_up = torch.cat([w.padded(prefix + n, ff, w.stride) for n in ("gate", "up")])
        self.w_down = w.padded(prefix + "down", w.stride, ff)
        self.b_gate_up = self.b_down = self.b_gate_up_f32 = None
        if self.bias:
            self.b_gate_up = torch.cat([w.vector(f"{prefix}{n}.b", ff, w.dtype)
                                        for n in ("gate", "up")])
            self.b_gate_up_f32 = self.b_gate_up.float()
            self.b_down = w.vector(prefix + "down.b", w.stride, w.dtype)

    def forward(self, h):
        if h.dtype != torch.float32 and h.shape[0] > self.MANY_ROWS:
            a = ops.group_gemm(h, self.w_gate_up, bias=self.b_gate_up_f32, act=self.act,
                               status=self.status)
        else:
            a = ops.gemm_act_mul(h, self.w_gate_up, self.act, bias=self.b_gate_up,
                                 status=self.status)
        return ops.gemm(a, self.w_down, bias=self.b_down, status=self.status), None


class MixtureOfExperts:
    """`top` of `experts` small feed-forwards per row, weighted by the softmax over the
    chosen logits, and an optional shared one.  Rows are sorted by expert; all experts of a
    product are one launch."""

    # rows per expert from which the rows are laid out by expert for the many-row product
    SORT_ROWS = 64

    def __init__(self, experts: int, top: int, ff: int, shared_ff: int | None,
                 act: int = _lib.ACT_SILU):
        if not 0 < top <= experts:
            raise ValueError(f"{top} of {experts} experts")
        self.experts, self.top, self.ff, self.act = experts, top, ff, act
        self.shared = GatedFeedForward(shared_ff, False, act) if shared_ff else None

    @staticmethod
    def tensor_shapes(prefix, width, experts, ff, shared_ff) -> dict:
        s = {prefix + "router": (experts, width), prefix + "router.b": (experts,)}
        for e in range(experts):
            s.update(GatedFeedForward.tensor_shapes(f"{prefix}e{e}.", width, ff, False))
        if shared_ff:
            s.update(GatedFeedForward.tensor_shapes(prefix + "shared.", width, shared_ff, False))
        return s

    @property
    def status(self):
        return self._status

    @status.setter
    def status(self, value):
        self._status = value
        if self.shared is not None:
            self.shared.status = value

    _status = None

    def load(self, w, prefix) -> None:
        ff = round_up(self.ff, 64)
        self.w_router = w.padded(prefix + "router", self.experts, w.stride)
        self.b_router = w.vector(prefix + "router.b")
        self.w_gate_up = w.zeros(self.experts, 2 * ff, w.stride)
        self.w_down = w.zeros(self.experts, w.stride, ff)
        for e in range(self.experts):
            p = f"{prefix}e{e}."
            self.w_gate_up[e, :self.ff, :w.width] = w.matrix(p + "gate")
            self.w_gate_up[e, ff:ff + self.ff, :w.width] = w.matrix(p + "up")
            self.w_down[e, :w.width, :self.ff] = w.matrix(p + "down")
        if self.shared is not None:
            self.shared.load(w, prefix + "shared.")

    def forward(self, h):
        z = ops.group_gemm(h, self.w_router, bias=self.b_router, out_f32=True,
                           status=self.status)
        r = ops.moe_route(z, self.top)
        each = -(-h.shape[0] * self.top // self.experts)
        x, gather = h, r.source
        if h.dtype != torch.float32 and each > self.SORT_ROWS:
            x, gather = ops.gather_rows(h, r.source, status=self.status), None
        a = ops.group_gemm(x, self.w_gate_up, offsets=r.offsets, gather=gather, act=self.act,
                           expect_rows=each, status=self.status)
        y = ops.group_gemm(a, self.w_down, offsets=r.offsets, expect_rows=each,
                           status=self.status)
        dense = self.shared.forward(h)[0] if self.shared is not None else None
        return dense, (y, r.place, r.share)
