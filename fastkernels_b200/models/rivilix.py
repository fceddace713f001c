"""Rivilix: a decoder whose mixer and feed-forward read the same residual row through a
layer norm each and are added side by side; mixers are a matrix memory (mLSTM) or latent
attention with YaRN rotation, feed-forwards dense with biases or a mixture of experts.  A
bigram embedding beside the token embedding, a soft cap on the logits, an fp32 residual, and
optionally a run of layers that is repeated with the same weights, each pass beginning with
x <- W [x; embedding output].

Per layer run, in launches:
  add_layernorm     outputs of the previous layer run added, both norms of the sum
  gemm              ONE projection for everything the mixer reads from its row
  latent attention  prepare, [query product, attention, merge, value product] or
                    [gather, expand, attention];  matrix memory: gates, step or units
  gemm              output projection
  gemm_act_mul, gemm  or  router, route, experts (two grouped products), shared expert
Rows are padded to 64 columns with zeros (weights have zero rows / columns there).
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch
import torch.nn as nn

from fastkernels_b200 import ops
from fastkernels_b200.infra.context import get_context
from fastkernels_b200.infra.tp import _tp_size

from .base import ServedModel
from .feedforward import GatedFeedForward, MixtureOfExperts
from .mixers import LatentAttention, MatrixMemory, Yarn, rope_table, round_up
from .weights import Packer, RandomSource


@dataclass
class MatrixMemoryConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass
class LatentConfig:
    heads: int
    dim: int
    rot: int
    vdim: int
    rank: int
    scale: float
    rot_base: float
    rot_scaling: Yarn | None = None


@dataclass
class DenseConfig:
    ff: int


@dataclass
class ExpertsConfig:
    experts: int
    top: int
    ff: int
    shared_ff: int | None = None


@dataclass
class RivilixLayer:
    mixer: MatrixMemoryConfig | LatentConfig
    ff: DenseConfig | ExpertsConfig | None       # None: no feed-forward


@dataclass
class Bigram:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass
class RivilixConfig:
    vocab_size: int
    hidden_size: int
    eps: float
    layers: list[RivilixLayer]
    loop: tuple[int, int, int] | None = None      # start, stop, times
    bigram: Bigram | None = None
    softcap: float | None = None
    dtype: torch.dtype = torch.bfloat16
    kv_block_size: int = 64
    order: list[tuple[int, bool]] = field(init=False)   # (layer, begins a pass) of every run

    def __post_init__(self):
        n = len(self.layers)
        self.order = [(i, False) for i in range(n)]
        if self.loop is not None:
            a, b, times = self.loop
            if not (0 <= a < b <= n and times >= 1):
                raise ValueError(f"loop {self.loop} does not fit {n} layers")
            body = [(i, i == a) for i in range(a, b)]
            self.order = self.order[:a] + body * times + self.order[b:]

    def tensor_shapes(self) -> dict:
        """Name -> shape of every weight."""
        w = self.hidden_size
        s = {"embed": (self.vocab_size, w), "final.norm": (w,), "final.norm.b": (w,),
             "head": (self.vocab_size, w)}
        if self.bigram is not None:
            s["bigram"] = (self.bigram.buckets + 1, w)
        if self.loop is not None:
            s["loop.in"] = (w, 2 * w)
        for i, layer in enumerate(self.layers):
            p, c, f = f"l{i}.", layer.mixer, layer.ff
            m = p + "mix."
            s.update({p + "norm1": (w,), p + "norm1.b": (w,)})
            if isinstance(c, MatrixMemoryConfig):
                hd, hv = c.heads * c.dim, c.heads * c.vdim
                s.update({m + "q": (hd, w), m + "k": (hd, w), m + "v": (hv, w), m + "g": (hv, w),
                          m + "o": (w, hv), m + "norm": (hv,)})
                for n in "if":
                    s.update({m + n: (c.heads, w), f"{m}{n}.b": (c.heads,)})
            else:
                s.update({m + "q": (c.heads * (c.dim + c.rot), w), m + "dkv": (c.rank + c.rot, w),
                          m + "dkv.norm": (c.rank,), m + "uk": (c.heads * c.dim, c.rank),
                          m + "uv": (c.heads * c.vdim, c.rank), m + "o": (w, c.heads * c.vdim)})
            if f is None:
                continue
            s.update({p + "norm2": (w,), p + "norm2.b": (w,)})
            if isinstance(f, DenseConfig):
                s.update(GatedFeedForward.tensor_shapes(p + "mlp.", w, f.ff, True))
            else:
                s.update(MixtureOfExperts.tensor_shapes(p + "mlp.", w, f.experts, f.ff,
                                                        f.shared_ff))
        return s


def _mixer_from_json(i: int, entry: dict):
    m = entry["mixer"]
    if entry["type"] == "mlstm":
        return MatrixMemoryConfig(m["heads"], m["dim"], m["vdim"], m["gate_cap"])
    if entry["type"] != "latent_attention":
        raise ValueError(f"layer {i}: unknown mixer '{entry['type']}'")
    rot = m.get("rot") or {}
    if rot.get("dims", m["rot_dim"]) != m["rot_dim"]:
        raise ValueError(f"layer {i}: the rotated part is rotated whole")
    y = rot.get("scaling")
    return LatentConfig(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["scale"],
                        rot.get("base", 1.0),
                        Yarn(y["factor"], y["original"], y["fast"], y["slow"]) if y else None)


def _ff_from_json(i: int, mlp: dict | None):
    if mlp is None:
        return None
    kind = mlp.get("kind", "dense")
    if kind == "dense":
        return DenseConfig(mlp["ff"])
    if kind != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward '{kind}'")
    shared = mlp.get("shared")
    return ExpertsConfig(mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"],
                         shared["ff"] if shared else None)


def config_from_json(cfg: dict, source, dtype=torch.bfloat16) -> RivilixConfig:
    layers = [RivilixLayer(_mixer_from_json(i, e), _ff_from_json(i, e.get("mlp")))
              for i, e in enumerate(cfg["layers"])]
    loop, big = cfg.get("loop"), (cfg.get("embedding") or {}).get("bigram")
    return RivilixConfig(
        vocab_size=cfg["vocab"], hidden_size=cfg["width"], eps=cfg["norm"]["eps"], layers=layers,
        loop=(loop["start"], loop["stop"], loop["times"]) if loop else None,
        bigram=Bigram(big["buckets"], big["mul_prev"], big["mul_cur"]) if big else None,
        softcap=cfg.get("logit_softcap"), dtype=dtype)


class _Layer:
    """Packed weights and sublayers of one layer."""

    def __init__(self, c: RivilixLayer, index: int, cfg: RivilixConfig):
        self.c, self.prefix = c, f"l{index}."
        m, f = c.mixer, c.ff
        if isinstance(m, MatrixMemoryConfig):
            self.mixer = MatrixMemory(m.heads, m.dim, m.vdim, m.gate_cap, cfg.eps, cfg.dtype)
        else:
            self.mixer = LatentAttention(m.heads, m.dim, m.rot, m.vdim, m.rank, m.scale,
                                         m.rot_base, m.rot_scaling, 0, cfg.eps, cfg.dtype)
        self.ff = None
        if isinstance(f, DenseConfig):
            self.ff = GatedFeedForward(f.ff, True)
        elif f is not None:
            self.ff = MixtureOfExperts(f.experts, f.top, f.ff, f.shared_ff)
        # columns of the mixer's projection, each section on a 16-byte boundary
        self.columns, at = {}, 0
        for name, n in self.mixer.sections.items():
            self.columns[name] = (at, at + n)
            at = round_up(at + n, 8)
        # per-head products read up to 15 columns beyond a section (against zero weights)
        self.in_rows = at + 16

    def load(self, w: Packer) -> None:
        p = self.prefix
        self.w_in = w.zeros(self.in_rows, w.stride)
        for name, m in self.mixer.load(w, p + "mix.").items():
            a, b = self.columns[name]
            self.w_in[a:b, :w.width] = m
        self.w_out = w.padded(self.mixer.pack_output(w.matrix(p + "mix.o")), w.stride,
                              self.mixer.out_columns)
        self.norm1 = w.vector(p + "norm1", w.stride), w.vector(p + "norm1.b", w.stride)
        self.norm2 = None
        if self.ff is not None:
            self.norm2 = w.vector(p + "norm2", w.stride), w.vector(p + "norm2.b", w.stride)
            self.ff.load(w, p + "mlp.")


class Rivilix(nn.Module, ServedModel):
    uses_state = True

    def __init__(self, config: RivilixConfig):
        super().__init__()
        if _tp_size() != 1:
            raise NotImplementedError("Rivilix is served on one GPU (no tensor parallelism)")
        if config.dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("Rivilix runs in bf16 or fp32")
        self.config = config
        self.device = torch.empty(0).device          # the default device in effect
        self.layers = [_Layer(c, i, config) for i, c in enumerate(config.layers)]
        # (layer, pass: which cache or state, begins a pass of the loop) of every run
        seen = [0] * len(self.layers)
        self.runs = []
        for i, begins in config.order:
            self.runs.append((i, seen[i], begins))
            seen[i] += 1
        self.passes = seen
        self.stride = round_up(config.hidden_size, 64)

    # ------------------------------------------------------------------ weights
    @torch.no_grad()
    def load_tensors(self, source) -> None:
        cfg = self.config
        w = Packer(source, self.device, cfg.dtype, cfg.hidden_size, self.stride)
        rows = round_up(cfg.vocab_size, 8)
        self.embed, self.head = (w.padded(n, rows, self.stride) for n in ("embed", "head"))
        self.pairs = None
        if cfg.bigram is not None:
            self.pairs = w.padded("bigram", cfg.bigram.buckets + 1, self.stride)
        self.w_loop = None
        if cfg.loop is not None:
            m = w.matrix("loop.in")
            self.w_loop = w.zeros(self.stride, 2 * self.stride)
            self.w_loop[:w.width, :w.width] = m[:, :w.width]
            self.w_loop[:w.width, self.stride:self.stride + w.width] = m[:, w.width:]
        self.final_norm = (w.vector("final.norm", self.stride),
                           w.vector("final.norm.b", self.stride))
        for layer in self.layers:
            layer.load(w)

    def init_random(self, seed, scale, rank=0):
        """Matrices randn * scale; norm weights 1, biases 0."""
        def init(name, shape, gen):
            if len(shape) == 2:
                return torch.empty(shape, dtype=self.config.dtype, device=self.device).normal_(
                    0.0, scale, generator=gen)
            return torch.full(shape, 0.0 if name.endswith(".b") else 1.0, dtype=torch.float32,
                              device=self.device)
        self.load_tensors(RandomSource(self.config.tensor_shapes(), init, seed, self.device))

    # ----------------------------------------------------------- caches and state
    def allocate_kv(self, num_blocks, block_size, device):
        pools = []
        for layer, passes in zip(self.layers, self.passes):
            if isinstance(layer.mixer, LatentAttention):
                pools += layer.mixer.allocate(passes, num_blocks[0], block_size, device)
        return pools

    def allocate_state(self, num_slots, device):
        self.last_ids = torch.zeros(num_slots, dtype=torch.int64, device=device)
        for layer, passes in zip(self.layers, self.passes):
            if isinstance(layer.mixer, MatrixMemory):
                layer.mixer.allocate(passes, num_slots, device)

    def preallocate(self, max_num_seqs, max_model_len, device, max_splits):
        self.status = ops.new_status(device) if torch.device(device).type == "cuda" else \
            torch.zeros(1, dtype=torch.int32)
        tables = {}
        for layer in self.layers:
            layer.mixer.status = self.status
            if layer.ff is not None:
                layer.ff.status = self.status
            if isinstance(layer.mixer, LatentAttention):
                m = layer.mixer
                key = m.rot, m.rot_base, m.rot_scaling
                if key not in tables:
                    tables[key] = rope_table(max_model_len, m.rot, m.rot_base, device,
                                             m.rot_scaling)
                m.cos_sin = tables[key]
        return self.status

    # -------------------------------------------------------------------- steps
    def forward(self, input_ids, positions):
        ctx, cfg = get_context(), self.config
        both = None                   # [x | embedding output] ahead of a pass of the loop
        if cfg.loop is not None:
            both = torch.empty((input_ids.shape[0], 2 * self.stride), dtype=cfg.dtype,
                               device=input_ids.device)
        pair = {}
        if cfg.bigram is not None:
            pair = dict(pairs=self.pairs, mul_prev=cfg.bigram.mul_prev,
                        mul_cur=cfg.bigram.mul_cur, last_ids=self.last_ids,
                        slots=ctx.state_slots, positions=positions, cu_portions=ctx.cu_portions)
        x = ops.embed_pair_f32(self.embed, input_ids, status=self.status,
                               copy=both[:, self.stride:] if both is not None else None, **pair)
        new = {}                      # what the layer run before adds to the residual
        for i, pass_no, begins in self.runs:
            layer = self.layers[i]
            if begins:
                ops.add_layernorm(x, cfg.hidden_size, cfg.eps, cfg.dtype, **new,
                                  out1=both[:, :self.stride], status=self.status)
                x, new = ops.group_gemm(both, self.w_loop, out_f32=True, status=self.status), {}
            x, h1, h2 = ops.add_layernorm(x, cfg.hidden_size, cfg.eps, cfg.dtype, **new,
                                          norm1=layer.norm1, norm2=layer.norm2,
                                          status=self.status)
            z = ops.gemm(h1, layer.w_in, status=self.status)
            cols = {name: z[:, a:b] for name, (a, b) in layer.columns.items()}
            y = layer.mixer.forward(h1, cols, positions, pass_no)
            new = {"a": ops.gemm(y, layer.w_out, status=self.status)}
            if layer.ff is not None:
                new["b"], new["experts"] = layer.ff.forward(h2)
        return ops.add_layernorm(x, cfg.hidden_size, cfg.eps, cfg.dtype, **new,
                                 norm1=self.final_norm, status=self.status)[1]

    def project(self, hidden):
        z = ops.gemm(hidden, self.head, status=self.status)[:, :self.config.vocab_size]
        return ops.softcap(z, self.config.softcap) if self.config.softcap else z

    @property
    def hidden_columns(self):
        return self.stride

    @property
    def logit_columns(self):
        return self.config.vocab_size


MODEL_CLASSES = {RivilixConfig: Rivilix}
