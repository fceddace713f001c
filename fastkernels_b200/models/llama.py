"""The Llama / Qwen3 dense decoders behind the engine's model interface."""
from __future__ import annotations

import torch

from fastkernels_b200 import ops
from fastkernels_b200.candidate.L4.llama import LlamaConfig, LlamaForCausalLM

from .base import ServedModel


class ServedLlama(LlamaForCausalLM, ServedModel):
    def __init__(self, config: LlamaConfig):
        if config.dtype != torch.bfloat16:
            raise ValueError("the Llama / Qwen3 decoders run in bf16 only")
        super().__init__(config)

    # ------------------------------------------------------------------ weights
    @torch.no_grad()
    def init_random(self, seed, scale, rank=0):
        """Random-init every parameter (randn * scale; norm weights 1.0).  Shards
        are drawn per rank: statistically the same model at every tp degree."""
        dev = next(self.parameters()).device
        g = torch.Generator(device=dev).manual_seed(seed * 1000003 + rank)
        for name, p in self.named_parameters():
            if "norm" in name or "layernorm" in name:
                p.fill_(1.0)
            else:
                p.normal_(0.0, scale, generator=g)

    @torch.no_grad()
    def load_full(self, w: dict) -> None:
        """UNSHARDED weights with merged qkv and gate_up matrices (l<i>.qkv, ...),
        through each parameter's weight_loader, which takes this rank's shard exactly
        as the reference loaders do."""
        c = self.config
        dev = next(self.parameters()).device

        def t(a):
            return torch.as_tensor(a).to(device=dev, dtype=c.dtype)

        emb = self.model.embed_tokens.embedding_op.emb.weight
        emb.weight_loader(emb, t(w["embed"]))
        lm = self.lm_head.embedding_op.emb.weight
        lm.weight_loader(lm, t(w["lm_head"]))
        self.model.norm.weight.copy_(t(w["norm"]))
        hq, hkv, d = c.num_attention_heads, c.num_key_value_heads, c.head_dim
        for li, layer in enumerate(self.model.layers):
            p = f"l{li}."
            layer.input_layernorm.weight.copy_(t(w[p + "ln1"]))
            layer.post_attention_layernorm.weight.copy_(t(w[p + "ln2"]))
            qkv = t(w[p + "qkv"])
            qp = layer.self_attn.qkv_proj.weight
            qp.weight_loader(qp, qkv[:hq * d], "q")
            qp.weight_loader(qp, qkv[hq * d:(hq + hkv) * d], "k")
            qp.weight_loader(qp, qkv[(hq + hkv) * d:], "v")
            op = layer.self_attn.o_proj.weight
            op.weight_loader(op, t(w[p + "o"]))
            gu = layer.mlp.gate_up_proj.weight
            gu.weight_loader(gu, t(w[p + "gate_up"]))
            dn = layer.mlp.down_proj.weight
            dn.weight_loader(dn, t(w[p + "down"]))
            if c.qk_norm:
                layer.self_attn.q_norm.weight.copy_(t(w[p + "qn"]))
                layer.self_attn.k_norm.weight.copy_(t(w[p + "kn"]))

    def load_tensors(self, source):
        """Hugging Face tensor names -> the merged layout of load_full."""
        w = {"embed": source.get("model.embed_tokens.weight"),
             "norm": source.get("model.norm.weight")}
        w["lm_head"] = source.get("lm_head.weight") if "lm_head.weight" in source else w["embed"]
        for i in range(self.config.num_hidden_layers):
            h, p = f"model.layers.{i}.", f"l{i}."
            att = h + "self_attn."
            w[p + "ln1"] = source.get(h + "input_layernorm.weight")
            w[p + "ln2"] = source.get(h + "post_attention_layernorm.weight")
            w[p + "qkv"] = torch.cat([source.get(f"{att}{s}_proj.weight") for s in "qkv"])
            w[p + "o"] = source.get(att + "o_proj.weight")
            w[p + "gate_up"] = torch.cat([source.get(f"{h}mlp.{s}_proj.weight")
                                          for s in ("gate", "up")])
            w[p + "down"] = source.get(h + "mlp.down_proj.weight")
            if self.config.qk_norm:
                w[p + "qn"] = source.get(att + "q_norm.weight")
                w[p + "kn"] = source.get(att + "k_norm.weight")
        self.load_full(w)

    # ----------------------------------------------------------------- KV cache
    def allocate_kv(self, num_blocks, block_size, device):
        """Pool [2, layers, num_blocks, BLOCK, Hkv/tp, D] (NHD) or
        [2, layers, num_blocks, Hkv/tp, BLOCK, D] (HND); every attention layer gets
        its K and V views (fastkernels/infra/engine.py:1783-1793)."""
        c = self.config
        hkv = self.model.layers[0].self_attn.num_kv_heads
        nb = num_blocks[0]
        shape = (nb, hkv, block_size, c.head_dim) if c.kv_layout == "HND" \
            else (nb, block_size, hkv, c.head_dim)
        kv = torch.zeros((2, c.num_hidden_layers, *shape), dtype=c.dtype, device=device)
        for li, layer in enumerate(self.model.layers):
            layer.self_attn.attn.k_cache = kv[0, li]
            layer.self_attn.attn.v_cache = kv[1, li]
        return kv

    def preallocate(self, max_num_seqs, max_model_len, device, max_splits):
        """One split-KV workspace serves every layer (they run back to back on one
        stream)."""
        for layer in self.model.layers:
            layer.self_attn.attn.decode_op._max_splits = max_splits
        first = self.model.layers[0].self_attn.attn.decode_op
        first.preallocate(max_num_seqs, device)
        ws_attr = "_fk_workspace" if hasattr(first, "_fk_workspace") else "_workspace"
        for layer in self.model.layers[1:]:
            op = layer.self_attn.attn.decode_op
            setattr(op, ws_attr, getattr(first, ws_attr))
            op._ws_batch, op._status = first._ws_batch, first._status
        self.attn_workspace = getattr(first, ws_attr)
        return first._status

    # -------------------------------------------------------------------- steps
    def begin_decode(self, ctx):
        """One split-KV schedule per step, shared by every layer."""
        att = self.model.layers[0].self_attn.attn
        op = att.decode_op
        ops.paged_decode_attn_plan(ctx.context_lens, ctx.block_tables, self.config.kv_block_size,
                                   att.num_heads, att.num_kv_heads, att.head_size,
                                   self.attn_workspace, op._max_splits, status=op._status)
        ctx.attn_plan_ready = True

    def project(self, hidden):
        return self.lm_head.project(hidden)

    def greedy(self, max_vals, max_idxs):
        return self.lm_head.greedy_pairs(max_vals, max_idxs)

    @property
    def hidden_columns(self):
        return self.config.hidden_size

    @property
    def logit_columns(self):
        return self.lm_head.per_partition


def config_from_json(cfg: dict, source, dtype) -> LlamaConfig:
    rope = cfg.get("rope_scaling") or {}
    heads = cfg["num_attention_heads"]
    if rope and rope.get("rope_type", rope.get("type", "default")) not in ("default", "llama3"):
        raise ValueError("only the default and llama3 RoPE scalings are served")
    return LlamaConfig(
        hidden_size=cfg["hidden_size"], intermediate_size=cfg["intermediate_size"],
        num_hidden_layers=cfg["num_hidden_layers"], num_attention_heads=heads,
        num_key_value_heads=cfg.get("num_key_value_heads", heads),
        head_dim=cfg.get("head_dim") or cfg["hidden_size"] // heads,
        vocab_size=cfg["vocab_size"],
        max_position_embeddings=cfg.get("max_position_embeddings", 8192),
        rms_norm_eps=cfg.get("rms_norm_eps", 1e-6), rope_theta=cfg.get("rope_theta", 10000.0),
        rope_scaling_factor=rope.get("factor", 1.0),
        rope_low_freq_factor=rope.get("low_freq_factor", 1.0),
        rope_high_freq_factor=rope.get("high_freq_factor", 1.0),
        rope_original_max_position_embeddings=rope.get("original_max_position_embeddings", 8192),
        dtype=dtype, qk_norm="model.layers.0.self_attn.q_norm.weight" in source)


MODEL_CLASSES = {LlamaConfig: ServedLlama}
