"""Prefill and decode throughput of the Pinuvik and Rivilix decoders beside decoders of the
same width, depth, heads and feed-forward (random weights, bf16), and the time of each
kernel of a layer beside its roofline.

    python bench.py --workload pinuvik|rivilix [--layers N] [--sizes 1b,8b] [--kernels]

pinuvik runs beside the Llama / Qwen3-style decoder, rivilix beside both.  A size is a
real model's layer; the number of layers is cut and the vocabulary is small.  Prefill runs whole prompts through the engine's
portion forward, decode replays the engine's CUDA graph; both are timed with CUDA
events on the launching stream.
"""
from __future__ import annotations

import json
import os

import numpy as np
import torch

from . import ops
from .candidate.L4.llama import LlamaConfig
from .engine import DecodeEngine
from .models.mixers import Yarn
from .models.pinuvik import PinuvikConfig, PinuvikLayer
from .models.rivilix import (Bigram, DenseConfig, ExpertsConfig, LatentConfig,
                             MatrixMemoryConfig, RivilixConfig, RivilixLayer)

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))

SIZES = {
    "1b": dict(width=2048, ff=6144, heads=16, kv=4, dim=128, chunk=1024, delta=(32, 64), rank=64),
    "3b-d64": dict(width=3072, ff=8192, heads=48, kv=12, dim=64, chunk=2048, delta=(24, 128),
                   rank=64),
    "8b": dict(width=4096, ff=12288, heads=32, kv=8, dim=128, chunk=2048, delta=(64, 64),
               rank=96),
}
# latent: heads, unrotated, rotated, value channels, rank; memory: heads, dim, vdim;
# experts: number, chosen, ff, shared ff
RIVILIX_SIZES = {
    "1b": dict(width=2048, ff=6144, latent=(16, 96, 32, 128, 512), memory=(8, 128, 256),
               experts=(32, 4, 1024, 2048), beside=dict(SIZES["1b"])),
    "3b-d64": dict(width=2560, ff=6400, latent=(40, 64, 32, 64, 256), memory=(10, 128, 256),
                   experts=(16, 2, 1600, 1600),
                   beside=dict(SIZES["3b-d64"], width=2560, ff=6400, heads=40, kv=10,
                               delta=(20, 128))),
    "8b": dict(width=4096, ff=12288, latent=(32, 96, 32, 128, 512), memory=(16, 128, 256),
               experts=(64, 6, 1408, 2816), beside=dict(SIZES["8b"])),
}
VOCAB = 32768
PREFILLS = [(1, 8192), (8, 1024)]
DECODES = [1, 16, 64]
CONTEXT = 1500
FP32_TFLOPS = 148 * 128 * 2 * 1.965e-3      # nominal fp32 rate outside the tensor cores


def peaks():
    p = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(p):
        with open(p) as f:
            return json.load(f)
    return {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}


def configs(z, layers):
    dh, dd = z["delta"]
    pin = PinuvikConfig(
        vocab_size=VOCAB, hidden_size=z["width"], eps=1e-6,
        layers=[PinuvikLayer(z["heads"], z["kv"], z["dim"], z["dim"] ** -0.5, z["chunk"],
                             z["dim"], 1e6, dh, dd, z["rank"], z["ff"])
                for _ in range(layers)])
    # the existing decoder has 128-channel heads only: same projection widths
    scale = 128 // z["dim"]
    llama = LlamaConfig(
        hidden_size=z["width"], intermediate_size=z["ff"], num_hidden_layers=layers,
        num_attention_heads=z["heads"] // scale, num_key_value_heads=z["kv"] // scale,
        head_dim=128, vocab_size=VOCAB, max_position_embeddings=16384, rope_theta=1e6,
        qk_norm=True, kv_block_size=64)
    return {"pinuvik": pin, "llama": llama}


def rivilix_configs(z, layers):
    """Half of the layers hold experts, every fourth a memory; the others' decoders as for
    `configs`."""
    h, dim, rot, vdim, rank = z["latent"]
    latent = LatentConfig(h, dim, rot, vdim, rank, (dim + rot) ** -0.5, 1e6,
                          Yarn(8.0, 4096, 32.0, 1.0))
    memory = MatrixMemoryConfig(*z["memory"], 15.0)
    dense, sparse = DenseConfig(z["ff"]), ExpertsConfig(*z["experts"])
    pattern = [RivilixLayer(memory, dense), RivilixLayer(latent, sparse),
               RivilixLayer(latent, dense), RivilixLayer(latent, sparse)]
    riv = RivilixConfig(vocab_size=VOCAB, hidden_size=z["width"], eps=1e-6,
                        layers=[pattern[i % 4] for i in range(layers)],
                        bigram=Bigram(8192, 40503, 9973), softcap=30.0)
    return {"rivilix": riv, **configs(z["beside"], layers)}


WORKLOADS = {"pinuvik": (SIZES, configs), "rivilix": (RIVILIX_SIZES, rivilix_configs)}


def _events():
    return torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)


def time_prefill(eng, n, length, iters=5):
    rs = np.random.RandomState(7)
    prompts = [rs.randint(0, VOCAB, size=length).tolist() for _ in range(n)]
    best = []
    for _ in range(iters + 2):
        seqs = [eng.open_sequence() for _ in range(n)]
        torch.cuda.synchronize()
        a, b = _events()
        a.record()
        hidden = eng._forward_portions([(s, 0, p) for s, p in zip(seqs, prompts)])
        eng.model.project(hidden[-1:])
        b.record()
        torch.cuda.synchronize()
        best.append(a.elapsed_time(b))
        for s in seqs:
            eng.finish(s)
    return float(np.median(best[2:]))


def time_decode(eng, batch, steps=32):
    """Every step's tokens are drawn anew: random weights would soon sample one and the
    same token in all sequences, and so visit few experts."""
    rs = np.random.RandomState(batch)
    eng.add_sequences([CONTEXT] * batch, list(range(batch)))

    def step():
        for s, t in zip(eng.seqs, rs.randint(0, VOCAB, size=batch).tolist()):
            s.last_token = t
        n = eng.prepare_decode(use_host_ids=True)
        bs = eng.graph_batch_size(n)
        eng.stage_inputs(n, bs, True)
        eng.run_step_device(bs)
        eng._mark_slot_in_flight()
        for s in eng.seqs:
            s.num_tokens += 1
    for _ in range(4):
        step()
    torch.cuda.synchronize()
    a, b = _events()
    a.record()
    for _ in range(steps):
        step()
    b.record()
    torch.cuda.synchronize()
    for s in list(eng.seqs):
        eng.finish(s)
    return a.elapsed_time(b) / steps


def _nbytes(*ts):
    return sum(t.numel() * t.element_size() for t in ts if torch.is_tensor(t))


def _work(name, args, kw, out):
    """(algorithmic bytes, tensor FLOPs) of one call."""
    t = list(args) + list(kw.values()) + (list(out) if isinstance(out, tuple) else [out])
    if name.startswith("gemm"):
        x, w = args[0], args[1]
        return _nbytes(x, w, out), 2 * x.shape[0] * w.shape[0] * w.shape[1]
    if name == "group_gemm":
        x, w, off = args[0], args[1], kw.get("offsets")
        wn, k = w.shape[-2:]
        rows, used = out.shape[0], 1 if w.dim() == 2 else w.shape[0]
        if off is not None:
            used = int((off[1:] > off[:-1]).sum().item())
        read = rows * k * (1 if off is not None else used) * 2
        return read + used * wn * k * 2 + _nbytes(out) if off is not None else \
            read + _nbytes(w) + rows * used * wn * out.element_size(), \
            2 * rows * wn * k * (1 if off is not None else used)
    if name == "latent_attn":
        q, lens, rank, rot = args[0], args[3].cpu().numpy(), args[7], args[8]
        qn = np.diff(args[2].cpu().numpy())
        pairs = float(sum((kv - n + 1 + kv) * n / 2 for n, kv in zip(qn, lens)))
        return int(lens.sum()) * (rank + rot) * 2 + _nbytes(q, out), \
            int(2 * pairs * q.shape[1] * (2 * rank + rot))
    if name == "mlstm_step":
        return _nbytes(*args[:3], args[4], out) + \
            2 * args[0].shape[0] * _nbytes(args[6][0], args[7][0]), 0
    if name == "mlstm_portions":
        q, k, v = args[:3]
        heads, dim, vdim = args[9:12]
        # what every block of 128 tokens adds to the state is written, read, replaced by the
        # state ahead of it and read again; both products with the matrix per token
        blocks = 4 * (q.shape[0] // 128) * heads * dim * vdim * 4
        return _nbytes(q, k, v, out) + blocks, 4 * q.shape[0] * heads * dim * vdim
    if name == "add_layernorm":
        ex = kw.get("experts")
        rows = _nbytes(kw.get("a"), kw.get("b"), *out[1:])
        gathered = ex[1].numel() * ex[0].shape[1] * ex[0].element_size() if ex else 0
        writes = _nbytes(args[0]) if kw.get("a") is not None else 0
        return _nbytes(args[0]) + writes + rows + gathered, 0
    if name == "embed_pair_f32":
        return 2 * _nbytes(out), 0
    if name in ("moe_route", "softcap"):
        return 2 * _nbytes(args[0]), 0
    if name == "latent_prepare":
        q, lat, out_q = args[0], args[1], args[8]
        return _nbytes(q, lat, lat) + (_nbytes(out_q) if args[10] else
                                       out_q.shape[0] * out_q.shape[1] * args[12] * 2), 0
    if name in ("latent_gather", "gather_rows"):
        return 2 * _nbytes(out), 0
    if name == "paged_decode_attn":
        q, k, lens = args[0], args[1], args[3]
        live = int(lens.sum().item())
        return 2 * live * k.shape[2] * k.shape[3] * 2 + 2 * _nbytes(q), 0
    if name == "prefill_attn":
        q, cu_q, cu_k = args[0], args[3].cpu().numpy(), args[4].cpu().numpy()
        pairs = sum((ck - cq + 1 + ck) * cq / 2 for cq, ck in zip(np.diff(cu_q), np.diff(cu_k)))
        return _nbytes(q, out) , int(4 * pairs * q.shape[1] * q.shape[2])
    if name == "rope_rms_store":
        return _nbytes(args[0], args[2]) + 3 * _nbytes(args[1]), 0
    if name == "qkv_rope_store":
        return 2 * _nbytes(args[0]), 0
    if name == "delta_scan":
        packed, state, cu, positions = args[0], args[1], args[2], args[4]
        # 4.25 fp32 multiply-adds per state element and token, on the fp32 pipes (not
        # tensor FLOPs: scaled so that the tensor peak below turns them into their time)
        fma = 4.25 * positions.numel() * state[0].numel()
        return _nbytes(packed, out) + 2 * (cu.numel() - 1) * _nbytes(state[0]), \
            2 * fma * peaks()["bf16_tflops"] / FP32_TFLOPS
    if name == "norm_shift":
        return _nbytes(args[0], kw.get("y"), out[1]) + \
            (_nbytes(args[0]) if kw.get("y") is not None else 0), 0
    if name == "branch_combine":
        return _nbytes(args[0], args[1], out) + 2 * _nbytes(args[5]), 0
    if name == "fused_add_rmsnorm":
        return 2 * _nbytes(args[0], args[1]), 0
    if name == "delta_prepare":
        return _nbytes(*args[:6], out), 0
    if name == "head_norm_gate":
        return _nbytes(args[0], args[1], out), 0
    if name == "embed_f32":
        return 2 * _nbytes(out), 0
    return _nbytes(*t), 0


OPS = ["gemm", "gemm_bf16", "gemm_act_mul", "gemm_silu_mul", "prefill_attn",
       "paged_decode_attn", "paged_decode_attn_plan", "rope_rms_store", "qkv_rope_store",
       "norm_shift", "branch_combine", "fused_add_rmsnorm", "rmsnorm", "delta_prepare",
       "delta_scan", "head_norm_gate", "act_and_mul", "silu_and_mul", "embed_f32",
       "group_gemm", "latent_attn", "latent_prepare", "latent_gather", "gather_rows",
       "mlstm_step", "mlstm_portions", "add_layernorm", "embed_pair_f32", "moe_route",
       "softcap"]


class OpTimer:
    """Times every op of one eager pass with event pairs.  Device work queued ahead
    (`preload`) keeps the host from being the clock."""

    def __init__(self):
        self.calls, self.depth, self.saved = [], 0, {}

    def __enter__(self):
        for name in OPS:
            fn = getattr(ops, name)
            self.saved[name] = fn

            def timed(*args, _fn=fn, _name=name, **kw):
                if self.depth:
                    return _fn(*args, **kw)
                self.depth += 1
                a, b = _events()
                a.record()
                out = _fn(*args, **kw)
                b.record()
                self.depth -= 1
                self.calls.append((_name, args, kw, out, a, b))
                return out
            setattr(ops, name, timed)
        return self

    def __exit__(self, *exc):
        for name, fn in self.saved.items():
            setattr(ops, name, fn)

    def table(self):
        torch.cuda.synchronize()
        pk, rows = peaks(), {}
        for name, args, kw, out, a, b in self.calls:
            nb, fl = _work(name, args, kw, out)
            label = name
            if name.startswith("gemm"):
                x, w = args[0], args[1]
                label += f" {x.shape[0]}x{w.shape[0]}x{w.shape[1]}"
            elif name == "group_gemm":
                label += f" {out.shape[0]}x" + "x".join(map(str, args[1].shape))
            r = rows.setdefault(label, [])
            floor = max(nb / pk["hbm_gbs"] / 1e6, fl / pk["bf16_tflops"] / 1e9)
            r.append((a.elapsed_time(b), floor))
        return {k: {"calls": len(v), "us": round(1e3 * float(np.median([t for t, _ in v])), 1),
                    "roofline_us": round(1e3 * float(np.median([f for _, f in v])), 1),
                    "frac": round(float(np.median([f / t for t, f in v])), 3)}
                for k, v in rows.items()}


def preload(ms_about=60.0):
    """Queue device work for about this long, so that the host runs ahead."""
    buf = torch.empty(4 << 30, dtype=torch.uint8, device="cuda")
    for _ in range(int(ms_about / 0.65)):
        ops.fill_u32(buf, 0)


def kernel_table(eng, n, length):
    """Per-op times of a prefill (length > 1) or decode (length == 1) pass."""
    rs = np.random.RandomState(7)
    if length > 1:
        prompts = [rs.randint(0, VOCAB, size=length).tolist() for _ in range(n)]
        for timed in (False, False, True):
            seqs = [eng.open_sequence() for _ in range(n)]
            if timed:
                preload()
                with OpTimer() as t:
                    eng._forward_portions([(s, 0, p) for s, p in zip(seqs, prompts)])
            else:
                eng._forward_portions([(s, 0, p) for s, p in zip(seqs, prompts)])
                for s in seqs:
                    eng.finish(s)
                torch.cuda.synchronize()
    else:
        eng.add_sequences([CONTEXT] * n, rs.randint(0, VOCAB, size=n).tolist())
        eng.prepare_decode(True)
        eng.stage_inputs(n, n, True)
        eng.enforce_eager = True
        for _ in range(2):           # kernels and allocations in place
            eng.run_step_device(n)
        eng.stage_inputs(n, n, True)
        torch.cuda.synchronize()
        preload()
        with OpTimer() as t:
            eng.run_step_device(n)
        eng.enforce_eager = False
        eng._mark_slot_in_flight()
    out = t.table()
    for s in list(eng.seqs):
        eng.finish(s)
    return out


def run(args, sampler=None):
    all_sizes, make = WORKLOADS[args.workload]
    sizes = args.sizes.split(",") if args.sizes else list(all_sizes)
    layers = args.layers or 8
    line = {"metric": f"{args.workload}_decoder_tokens_per_s", "unit": "tok/s", "dtype": "bf16",
            "data": "synthetic", "n_gpus": 1, "layers": layers, "vocab": VOCAB,
            "context": CONTEXT, "sizes": {}}
    if sampler:
        sampler.start()
    for name in sizes:
        z, res = all_sizes[name], {}
        for kind, cfg in make(z, layers).items():
            tokens = max(n * t for n, t in PREFILLS)
            pages = max(tokens // 64 + 64, max(DECODES) * (2048 // 64 + 1) + 64)
            eng = DecodeEngine(cfg, max_num_seqs=max(DECODES), max_model_len=16384,
                               num_kv_blocks=pages, init_scale=0.02)
            r = {}
            for n, t in PREFILLS:
                ms = time_prefill(eng, n, t)
                r[f"prefill {n}x{t}"] = {"ms": round(ms, 3), "tok_s": round(n * t / ms * 1e3)}
            eng.capture_cudagraph(DECODES)
            for b in DECODES:
                ms = time_decode(eng, b)
                r[f"decode batch {b}"] = {"ms": round(ms, 4), "tok_s": round(b / ms * 1e3)}
            if args.kernels:
                r["kernels prefill 1x8192"] = kernel_table(eng, 1, 8192)
                r["kernels prefill 8x1024"] = kernel_table(eng, 8, 1024)
                r["kernels decode batch 64"] = kernel_table(eng, 64, 1)
            r["device_status_word"] = eng.device_status()
            res[kind] = r
            eng.graphs.clear()
            del eng
            torch.cuda.empty_cache()
        line["sizes"][name] = {"config": z, **res}
    if sampler:
        line["clocks"] = sampler.stop()
    print(json.dumps(line), flush=True)
