"""Pinuvik: a decoder with two mixers side by side in every layer (chunked rotary
attention and a generalized delta rule), sandwich norms with one gain each, a token
shift ahead of the mixers, an fp32 residual stream and an optional run of layers that
is repeated with the same weights.

Per layer run, in launches:
  norm_shift        previous feed-forward's output normed into the residual, norm,
                    token shift
  gemm              ONE projection for everything both mixers read from the row
  rope_rms_store / attention          delta_prepare / delta_scan / head_norm_gate
  gemm x 2          the two output projections
  branch_combine    their norms, half-sum, norm, residual, norm of the feed-forward
  gemm_act_mul, gemm
Rows are padded to 64 columns with zeros (weights have zero rows / columns there).
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch
import torch.nn as nn

from fastkernels_b200 import _lib, ops
from fastkernels_b200.infra.context import get_context
from fastkernels_b200.infra.tp import _tp_size

from .base import ServedModel
from .mixers import GeneralizedDelta, RotaryAttention, rope_table, round_up
from .weights import RandomSource


@dataclass
class PinuvikLayer:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    chunk: int | None            # tokens per attention chunk, None = whole context
    rot_dims: int
    rot_base: float
    delta_heads: int
    delta_dim: int
    decay_rank: int
    ff: int | None               # None: no feed-forward


@dataclass
class PinuvikConfig:
    vocab_size: int
    hidden_size: int
    eps: float
    layers: list[PinuvikLayer]
    loop: tuple[int, int, int] | None = None      # start, stop, times
    dtype: torch.dtype = torch.bfloat16
    kv_block_size: int = 64
    order: list[int] = field(init=False)          # layer index of every run

    def __post_init__(self):
        n = len(self.layers)
        self.order = list(range(n))
        if self.loop is not None:
            a, b, times = self.loop
            if not (0 <= a <= b <= n and times >= 0):
                raise ValueError(f"loop {self.loop} does not fit {n} layers")
            self.order = self.order[:a] + self.order[a:b] * times + self.order[b:]

    def tensor_shapes(self) -> dict:
        """Name -> shape of every weight."""
        w = self.hidden_size
        s = {"embed": (self.vocab_size, w), "final.norm": (), "head": (self.vocab_size, w)}
        for i, c in enumerate(self.layers):
            p = f"l{i}."
            s.update({p + "norm1": (), p + "norm1b": (), p + "shift": (w,)})
            left, right, hd = p + "mix.left.", p + "mix.right.", c.delta_heads * c.delta_dim
            s.update({left + "q": (c.heads * c.dim, w), left + "k": (c.kv_heads * c.dim, w),
                      left + "o": (w, c.heads * c.dim), left + "out": (w,)})
            s.update({right + x: (hd, w) for x in "rkvga"})
            s.update({right + "a.b": (hd,), right + "w0": (hd,), right + "norm": (hd,),
                      right + "w1": (c.decay_rank, w), right + "w2": (hd, c.decay_rank),
                      right + "o": (w, hd), right + "out": (w,)})
            if c.ff is not None:
                s.update({p + "norm2": (), p + "norm2b": (), p + "mlp.gate": (c.ff, w),
                          p + "mlp.up": (c.ff, w), p + "mlp.down": (w, c.ff)})
        return s


def config_from_json(cfg: dict, source, dtype=torch.bfloat16) -> PinuvikConfig:
    """config.json -> PinuvikConfig; the rank of the decay's low-rank pair is the only
    size that a tensor's shape gives (`source`: the folder's tensors)."""
    layers = []
    for i, entry in enumerate(cfg["layers"]):
        if entry["type"] != "parallel":
            raise ValueError(f"layer {i}: unknown mixer '{entry['type']}'")
        left, right = entry["mixer"]["left"], entry["mixer"]["right"]
        if left.get("vdim", left["dim"]) != left["dim"]:
            raise ValueError(f"layer {i}: values are the keys, so vdim must equal dim")
        mlp = entry.get("mlp")
        if mlp is not None and mlp.get("kind", "dense") != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward '{mlp['kind']}'")
        mask, rot = left.get("mask") or {}, left.get("rot") or {}
        layers.append(PinuvikLayer(
            heads=left["heads"], kv_heads=left.get("kv_heads", left["heads"]), dim=left["dim"],
            scale=left["scale"], chunk=mask.get("size"), rot_dims=rot.get("dims", 0),
            rot_base=rot.get("base", 1.0), delta_heads=right["heads"], delta_dim=right["dim"],
            decay_rank=source.shape(f"l{i}.mix.right.w1")[0],
            ff=None if mlp is None else mlp["ff"]))
    loop = cfg.get("loop")
    return PinuvikConfig(
        vocab_size=cfg["vocab"], hidden_size=cfg["width"], eps=cfg["norm"]["eps"], layers=layers,
        loop=(loop["start"], loop["stop"], loop["times"]) if loop else None, dtype=dtype)


class _Layer:
    """Packed weights and mixers of one layer."""

    def __init__(self, c: PinuvikLayer, index: int, cfg: PinuvikConfig, span: int):
        self.cfg, self.c, self.prefix = cfg, c, f"l{index}."
        self.left = RotaryAttention(c.heads, c.kv_heads, c.dim, c.scale, c.rot_dims, c.rot_base,
                                    span, cfg.eps, cfg.dtype)
        self.right = GeneralizedDelta(c.delta_heads, c.delta_dim, c.decay_rank, cfg.eps,
                                      cfg.dtype)
        # columns of the shared projection, each section on a 16-byte boundary
        self.columns, at = {}, 0
        for side, mixer in (("left", self.left), ("right", self.right)):
            for name, n in mixer.sections.items():
                self.columns[side, name] = (at, at + n)
                at = round_up(at + n, 8)
        self.in_rows = at

    def load(self, source, device) -> None:
        cfg, c, p = self.cfg, self.c, self.prefix
        stride = round_up(cfg.hidden_size, 64)

        def weight(name):
            return source.get(name).to(device=device, dtype=cfg.dtype)

        def vector(name, pad=None):
            v = source.get(name).to(device=device, dtype=torch.float32).reshape(-1)
            if pad is None:
                return v.contiguous()
            out = torch.zeros(pad, dtype=torch.float32, device=device)
            out[:v.numel()] = v
            return out

        def padded(w, rows, cols):
            out = torch.zeros((rows, cols), dtype=cfg.dtype, device=device)
            out[:w.shape[0], :w.shape[1]] = w
            return out

        self.w_in = torch.zeros((self.in_rows, stride), dtype=cfg.dtype, device=device)
        for (side, name), (a, b) in self.columns.items():
            self.w_in[a:b, :cfg.hidden_size] = weight(f"{p}mix.{side}.{name}")
        self.w_left = padded(self.left.pack_output(weight(p + "mix.left.o")), stride,
                             self.left.out_columns)
        self.w_right = padded(self.right.pack_output(weight(p + "mix.right.o")), stride,
                              self.right.out_columns)
        self.out_left = vector(p + "mix.left.out", stride)
        self.out_right = vector(p + "mix.right.out", stride)
        r, right = p + "mix.right.", self.right
        hd = c.delta_heads * c.delta_dim
        right.w2 = padded(weight(r + "w2"), hd, round_up(c.decay_rank, 4))
        right.w0, right.a_bias = vector(r + "w0"), vector(r + "a.b")
        right.norm = vector(r + "norm")
        self.norm1, self.norm1b = vector(p + "norm1"), vector(p + "norm1b")
        self.shift = vector(p + "shift", stride)
        self.norm2 = self.norm2b = None
        if c.ff is not None:
            self.norm2, self.norm2b = vector(p + "norm2"), vector(p + "norm2b")
            ff = round_up(c.ff, 64)
            self.w_gate_up = torch.cat([padded(weight(p + "mlp.gate"), ff, stride),
                                        padded(weight(p + "mlp.up"), ff, stride)])
            self.w_down = padded(weight(p + "mlp.down"), stride, ff)


class Pinuvik(nn.Module, ServedModel):
    uses_state = True

    def __init__(self, config: PinuvikConfig):
        super().__init__()
        if _tp_size() != 1:
            raise NotImplementedError("Pinuvik is served on one GPU (no tensor parallelism)")
        if config.dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("Pinuvik runs in bf16 or fp32")
        self.config = config
        self.device = torch.empty(0).device          # the default device in effect
        spans = self.spans_of(config)
        self.layers = [_Layer(c, i, config, spans.index(c.chunk))
                       for i, c in enumerate(config.layers)]
        # pass number of every run of a layer: which pool it uses
        seen = [0] * len(self.layers)
        self.runs = []
        for i in config.order:
            self.runs.append((i, seen[i]))
            seen[i] += 1
        self.passes = seen
        self.stride = round_up(config.hidden_size, 64)

    @classmethod
    def spans_of(cls, config):
        return sorted({c.chunk for c in config.layers}, key=lambda x: (x is None, x or 0))

    # ------------------------------------------------------------------ weights
    @torch.no_grad()
    def load_tensors(self, source) -> None:
        cfg, dev = self.config, self.device

        def table(name):
            w = torch.zeros((round_up(cfg.vocab_size, 8), self.stride), dtype=cfg.dtype,
                            device=dev)
            w[:cfg.vocab_size, :cfg.hidden_size] = source.get(name).to(device=dev,
                                                                       dtype=cfg.dtype)
            return w

        self.embed, self.head = table("embed"), table("head")
        self.final_norm = source.get("final.norm").to(device=dev, dtype=torch.float32).reshape(-1)
        for layer in self.layers:
            layer.load(source, dev)

    def init_random(self, seed, scale, rank=0):
        """Matrices randn * scale; norm gains and weights 1, shift 1/2, biases 0."""
        def init(name, shape, gen):
            leaf = name.rsplit(".", 1)[-1]
            if len(shape) == 2:
                return torch.empty(shape, dtype=self.config.dtype, device=self.device).normal_(
                    0.0, scale, generator=gen)
            value = {"shift": 0.5, "b": 0.0, "w0": 0.0}.get(leaf, 1.0)
            return torch.full(shape, value, dtype=torch.float32, device=self.device)
        self.load_tensors(RandomSource(self.config.tensor_shapes(), init, seed, self.device))

    # ----------------------------------------------------------- caches and state
    def allocate_kv(self, num_blocks, block_size, device):
        pools = []
        for layer, passes in zip(self.layers, self.passes):
            pools += layer.left.allocate(passes, num_blocks[layer.left.span], block_size, device)
        return pools

    def allocate_state(self, num_slots, device):
        for layer, passes in zip(self.layers, self.passes):
            layer.right.allocate(passes, num_slots, device)
        self.shift_state = torch.zeros((len(self.runs), num_slots, self.stride),
                                       dtype=torch.float32, device=device)

    def preallocate(self, max_num_seqs, max_model_len, device, max_splits):
        self.status = ops.new_status(device) if torch.device(device).type == "cuda" else \
            torch.zeros(1, dtype=torch.int32)
        self.num_sms = torch.cuda.get_device_properties(device).multi_processor_count \
            if torch.device(device).type == "cuda" else 1
        tables = {}
        self.plans = {}            # (span, query heads, KV heads) -> workspace
        for layer in self.layers:
            att = layer.left
            key = att.rot_dims, att.rot_base
            if key not in tables:
                tables[key] = rope_table(max_model_len, *key, device)
            att.cos_sin = tables[key]
            att.status = layer.right.status = self.status
            if not att.tensor_cores:
                continue
            longest = max_model_len if layer.c.chunk is None else min(layer.c.chunk,
                                                                      max_model_len)
            att.max_splits = min(max_splits, ops.max_splits_for(longest))
            if att.plan_key not in self.plans:
                n = ops.attn_workspace_bytes(max_num_seqs, att.kv_heads * att.group,
                                             att.padded_dim, att.max_splits)
                self.plans[att.plan_key] = (torch.empty(n, dtype=torch.uint8, device=device),
                                            att)
            att.workspace = self.plans[att.plan_key][0]
        return self.status

    # -------------------------------------------------------------------- steps
    def begin_decode(self, ctx):
        """One split-KV schedule per span and head layout, shared by its layers; small
        steps need none (their attention is a single self-planning launch)."""
        planned = {}
        for key, (workspace, att) in self.plans.items():
            span = ctx.spans[att.span]
            n, block = span.block_tables.shape[0], self.config.kv_block_size
            if n * att.kv_heads <= self.num_sms and span.block_tables.stride(0) * block <= 2048:
                planned[key] = False
                continue
            ops.paged_decode_attn_plan(span.kv_lens, span.block_tables, block,
                                       att.kv_heads * att.group, att.kv_heads, att.padded_dim,
                                       workspace, att.max_splits, status=self.status)
            planned[key] = True
        for layer in self.layers:
            layer.left.plan = planned.get(layer.left.plan_key, False)

    def forward(self, input_ids, positions):
        ctx, cfg = get_context(), self.config
        x = ops.embed_f32(self.embed, input_ids, status=self.status)
        y = y_gain = None
        for run, (i, pass_no) in enumerate(self.runs):
            layer = self.layers[i]
            x, h = ops.norm_shift(x, layer.norm1, cfg.hidden_size, cfg.eps, cfg.dtype, y=y,
                                  y_gain=y_gain, shift=layer.shift,
                                  state=self.shift_state[run], slots=ctx.state_slots,
                                  positions=positions, cu_portions=ctx.cu_portions,
                                  status=self.status)
            z = ops.gemm(h, layer.w_in, status=self.status)
            cols = {"left": {}, "right": {}}
            for (side, name), (a, b) in layer.columns.items():
                cols[side][name] = z[:, a:b]
            left = ops.gemm(layer.left.forward(cols["left"], positions, pass_no), layer.w_left,
                            status=self.status)
            right = ops.gemm(layer.right.forward(cols["right"], positions, pass_no),
                             layer.w_right, status=self.status)
            h = ops.branch_combine(left, right, layer.out_left, layer.out_right, layer.norm1b, x,
                                   cfg.hidden_size, cfg.eps, gain=layer.norm2)
            y = y_gain = None
            if layer.c.ff is not None:
                act = ops.gemm_act_mul(h, layer.w_gate_up, _lib.ACT_GELU_TANH,
                                       status=self.status)
                y, y_gain = ops.gemm(act, layer.w_down, status=self.status), layer.norm2b
        return ops.norm_shift(x, self.final_norm, cfg.hidden_size, cfg.eps, cfg.dtype, y=y,
                              y_gain=y_gain, status=self.status)[1]

    def project(self, hidden):
        return ops.gemm(hidden, self.head, status=self.status)[:, :self.config.vocab_size]

    @property
    def hidden_columns(self):
        return self.stride

    @property
    def logit_columns(self):
        return self.config.vocab_size


MODEL_CLASSES = {PinuvikConfig: Pinuvik}
