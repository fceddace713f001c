"""Serving engine: paged KV pools, recurrent-state slots, prefill in portions,
CUDA-graph decode, greedy sampling, tensor parallelism (one process per GPU, NCCL).
The model behind it is chosen by its configuration (models.registry).

Mirror of the decode path of the reference engine (fastkernels/infra/engine.py):
  BlockManager.maybe_append_pages            engine.py:530-537
  ModelRunner.allocate_kv_cache              engine.py:1783-1793  (pool layout)
  ModelRunner._prepare_decode_arrays         engine.py:5767-5838  (positions / slots / lens)
  ModelRunner._run_graph_from_numpy          engine.py:5386-5427  (H2D staging + replay)
  ModelRunner.capture_cudagraph              engine.py:6701-7025  (graph body, graph_vars)
  ModelRunner._greedy_from_hidden            engine.py:5711-5746  (argmax, tp all-gather)
plus the prefill side of ModelRunner.run (engine.py:4902-4990, 6048-6063): whole
or chunked prompts fill their KV pages and join the running batch.  `feed` runs
given tokens of any mix of sequences (portions of prompts and single tokens) and
returns logits.  HTTP serving is outside this build; sequences may also enter with
their context already in the cache (synthetic contexts for the benchmark, or
whatever the caller wrote).

Every rank of a tensor-parallel group runs this same host code on the same
inputs (deterministic scheduling), so no control-plane exchange is needed; the
data-path exchanges are the NCCL all-reduces after o_proj / down_proj / the
vocab-parallel embedding and the (max, index) all-gather of greedy sampling,
all captured in the CUDA graph.
"""
from __future__ import annotations

import os

import numpy as np
import torch

from . import ops
from .cache import BlockManager, Sequence, StateSlots, pack_prefill_chunk
from .infra.context import SpanBatch, get_context, reset_context, set_context
from .infra.tp import _tp_rank, _tp_size
from .models.registry import load_folder, model_class

# FK_B200_PREPARE_AHEAD=0: stage every step's host arrays only when the step is
# called (for A/B timing of the look-ahead in DecodeEngine.step)
_NO_PREPARE_AHEAD = os.environ.get("FK_B200_PREPARE_AHEAD", "1") == "0"


class DecodeEngine:
    def __init__(self, config, *, max_num_seqs: int, max_model_len: int,
                 num_kv_blocks: int | list[int], device="cuda", seed: int = 0,
                 enforce_eager: bool = False, init_scale: float | None = 0.02,
                 attn_max_splits: int | None = None):
        """num_kv_blocks: pages of the KV pool, one number for every span of the model
        or one per span.  init_scale None leaves the weights for load_weights."""
        self.config = config
        self.device = torch.device(device)
        self.tp, self.rank = _tp_size(), _tp_rank()
        self.block_size = config.kv_block_size
        self.max_num_seqs = max_num_seqs
        self.max_model_len = max_model_len
        self.enforce_eager = enforce_eager
        self.h2d_bytes = 0
        self.d2h_bytes = 0

        prev = torch.get_default_dtype()
        torch.set_default_dtype(config.dtype)
        try:
            with torch.device(self.device):
                self.model = model_class(config)(config)
        finally:
            torch.set_default_dtype(prev)
        if init_scale is not None:
            self.init_random_weights(seed, init_scale)
        if attn_max_splits is None:
            attn_max_splits = ops.max_splits_for(max_model_len)
        self._attn_max_splits = attn_max_splits

        # tensor parallel: fused all-reduce + add + RMSNorm over peer memory unless
        # FK_B200_NCCL_ALLREDUCE=1 asks for the plain NCCL path
        self.comm = None
        if self.tp > 1 and self.device.type == "cuda" and \
                os.environ.get("FK_B200_NCCL_ALLREDUCE", "0") != "1":
            from .comm import TpComm, set_tp_comm
            # rows: one prefill chunk (512, the most a fused call takes); a decode
            # batch has to fit the same limit
            if max_num_seqs > 512:
                raise ValueError("tensor-parallel decode batches are limited to 512 sequences "
                                 "by the fused all-reduce (set FK_B200_NCCL_ALLREDUCE=1 for more)")
            self.comm = TpComm(512, self.model.hidden_columns, self.device)
            algo = os.environ.get("FK_B200_ALLREDUCE_ALGO", "auto")
            if algo not in ("auto", "one_stage", "two_stage", "push"):
                raise ValueError("FK_B200_ALLREDUCE_ALGO must be auto, one_stage, two_stage "
                                 "or push")
            self.comm.algo = algo
            set_tp_comm(self.comm)
        spans = self.model.kv_spans
        per_span = list(num_kv_blocks) if isinstance(num_kv_blocks, (list, tuple)) \
            else [num_kv_blocks] * len(spans)
        self.span_blocks = [BlockManager(nb, self.block_size, g, chunk)
                            for g, (nb, chunk) in enumerate(zip(per_span, spans))]
        self.blocks = self.span_blocks[0]
        self.max_num_blocks = [b.max_blocks(max_model_len) for b in self.span_blocks]
        self.allocate_kv_cache(per_span)
        self.state_slots = StateSlots(max_num_seqs) if self.model.uses_state else None
        if self.state_slots is not None:
            self.model.allocate_state(max_num_seqs, self.device)
        self.seqs: list[Sequence] = []
        self._next_id = 0
        self._init_buffers()
        self.graphs: dict[int, torch.cuda.CUDAGraph] = {}
        self.graph_pool = None
        self._bt_dirty = True
        self._staged_for = None     # ids of the sequences the device tables belong to

    @staticmethod
    def pages_for(config, max_tokens: int, max_num_seqs: int) -> list[int]:
        """Pages per span that hold max_tokens tokens of up to max_num_seqs sequences:
        whole pages, and one more for the last page of every sequence and of every chunk
        (a portion keeps all the pages it touches until it has run)."""
        return [-(-max_tokens // config.kv_block_size) + max_num_seqs
                + (0 if chunk is None else max_tokens // chunk + 1)
                for chunk in model_class(config).spans_of(config)]

    @classmethod
    def from_folder(cls, folder, *, max_tokens: int, max_num_seqs: int, dtype=torch.bfloat16,
                    **kw):
        """Engine for the model in a folder (config.json, safetensors), with pages for
        max_tokens live tokens in all."""
        config, source = load_folder(folder, dtype)
        eng = cls(config, init_scale=None, max_num_seqs=max_num_seqs,
                  max_model_len=max_tokens + 1,
                  num_kv_blocks=cls.pages_for(config, max_tokens, max_num_seqs), **kw)
        eng.load_weights(source)
        return eng

    # ------------------------------------------------------------------ weights
    def init_random_weights(self, seed: int, scale: float) -> None:
        self.model.init_random(seed, scale, self.rank)

    @torch.no_grad()
    def load_weights(self, source) -> None:
        """Weights from a models.weights.TensorSource."""
        self.model.load_tensors(source)

    def load_full_weights(self, w: dict) -> None:
        """UNSHARDED Llama / Qwen3 weights in the merged layout of ServedLlama.load_full."""
        self.model.load_full(w)

    # ----------------------------------------------------------------- KV cache
    def allocate_kv_cache(self, num_blocks) -> None:
        """Page pools of all spans, installed into the attention layers; kv_cache is
        what the model returns (one tensor [2, layers, ...] where all layers share a
        shape)."""
        per_span = list(num_blocks) if isinstance(num_blocks, (list, tuple)) \
            else [num_blocks] * len(self.span_blocks)
        self.num_kv_blocks = per_span[0]
        self.kv_cache = self.model.allocate_kv(per_span, self.block_size, self.device)

    @torch.no_grad()
    def fill_kv_random(self, seed: int, scale: float = 0.5) -> None:
        """Synthetic contexts: fill the whole pool with randn * scale."""
        g = torch.Generator(device=self.device).manual_seed(seed * 7919 + self.rank)
        pools = self.kv_cache if isinstance(self.kv_cache, (list, tuple)) \
            else [self.kv_cache[:, li] for li in range(self.kv_cache.shape[1])]
        for pool in pools:
            pool.normal_(0.0, scale, generator=g)

    # ------------------------------------------------------------------ buffers
    def _init_buffers(self) -> None:
        n, dev, c = self.max_num_seqs, self.device, self.config
        nsp = len(self.span_blocks)
        # The per-step inputs live in ONE buffer, [input_ids i64 | positions i64 |
        # (slot_mapping i32 | context_lens i32) per span | state slots i32], so that a
        # step stages them with a single host-to-device copy (all of it, or all but the
        # token ids when those stay on the device).
        self._packed_bytes = n * (16 + 8 * nsp + (4 if self.state_slots is not None else 0))

        def packed_views(buf):
            v = dict(input_ids=buf[:8 * n].view(torch.int64),
                     positions=buf[8 * n:16 * n].view(torch.int64))
            slots, lens, o = [], [], 16 * n
            for _ in range(nsp):
                slots.append(buf[o:o + 4 * n].view(torch.int32))
                lens.append(buf[o + 4 * n:o + 8 * n].view(torch.int32))
                o += 8 * n
            v.update(slot_mapping=slots[0], context_lens=lens[0], span_slots=slots,
                     span_lens=lens)
            if self.state_slots is not None:
                v["state_slots"] = buf[o:o + 4 * n].view(torch.int32)
            return v

        def clear(v):
            for t in v["span_slots"]:
                t.fill_(-1)                     # no slot
            if "state_slots" in v:
                v["state_slots"].fill_(-1)

        self._packed_dev = torch.zeros(self._packed_bytes, dtype=torch.uint8, device=dev)
        tables = [torch.full((n, cols), -1, dtype=torch.int32, device=dev)
                  for cols in self.max_num_blocks]
        self.graph_vars = dict(
            **packed_views(self._packed_dev),
            block_tables=tables[0], span_tables=tables,
            outputs=torch.zeros((n, self.model.hidden_columns), dtype=c.dtype, device=dev),
            lm_logits=torch.zeros((n, self.model.logit_columns), dtype=c.dtype, device=dev),
            lm_max_vals=torch.zeros(n, dtype=torch.float32, device=dev),
            lm_max_idxs=torch.zeros(n, dtype=torch.int64, device=dev),
            token_ids=torch.zeros(n, dtype=torch.int64, device=dev),
            cu_rows=torch.arange(n + 1, dtype=torch.int32, device=dev),
        )
        clear(self.graph_vars)

        def pinned(shape, dtype):
            return torch.zeros(shape, dtype=dtype).pin_memory() if dev.type == "cuda" \
                else torch.zeros(shape, dtype=dtype)

        # Ring of pinned staging slots: an async H2D copy reads the pinned buffer
        # when the copy EXECUTES, so a slot may be rewritten only after the copies
        # issued from it have completed (the slot's event).  The host can therefore
        # run up to RING - 1 steps ahead of the device.
        self.RING = 4
        self._ring = []
        for _ in range(self.RING):
            packed = pinned(self._packed_bytes, torch.uint8)
            tables = [pinned((n, cols), torch.int32) for cols in self.max_num_blocks]
            slot = dict(**packed_views(packed), packed=packed, block_tables=tables[0],
                        span_tables=tables, token_ids=pinned(n, torch.int64))
            clear(slot)
            self._ring.append(slot)
        self._ring_np = [{k: [t.numpy() for t in v] if isinstance(v, list) else v.numpy()
                          for k, v in slot.items()} for slot in self._ring]
        self._ring_events = [None] * self.RING
        self._ring_pos = 0
        # (sequence-set version, count) the staging slot was prepared ahead for, or None
        self._ahead = None
        self._seq_epoch = 0
        self.host, self.host_np = self._ring[0], self._ring_np[0]
        self.status = self.model.preallocate(n, self.max_model_len, dev, self._attn_max_splits)
        self.attn_workspace = getattr(self.model, "attn_workspace", None)

    # ---------------------------------------------------------------- sequences
    def _new_sequence(self, num_tokens: int, last_token: int = 0) -> Sequence:
        s = Sequence(self._next_id, num_tokens, last_token=last_token)
        self._next_id += 1
        if self.state_slots is not None:
            self.state_slots.allocate(s)
        return s

    def _running_set_changed(self) -> None:
        self._bt_dirty = True
        self._seq_epoch += 1
        self._ahead = None

    def add_sequences(self, context_lens, first_tokens) -> list[Sequence]:
        """Register running sequences whose first `L - 1` tokens are already in
        the cache and whose L-th token (`first_tokens[i]`) is the next input."""
        out = []
        for L, tok in zip(context_lens, first_tokens):
            if len(self.seqs) >= self.max_num_seqs:
                raise RuntimeError("max_num_seqs exceeded")
            if L < 1 or L > self.max_model_len:
                raise ValueError(f"context length {L} outside [1, {self.max_model_len}]")
            s = self._new_sequence(int(L), int(tok))
            for blocks in self.span_blocks:
                blocks.allocate(s)
            self.seqs.append(s)
            out.append(s)
        self._running_set_changed()
        return out

    def open_sequence(self) -> Sequence:
        """A running sequence without tokens; they come through feed()."""
        if len(self.seqs) >= self.max_num_seqs:
            raise RuntimeError("max_num_seqs exceeded")
        s = self._new_sequence(0)
        self.seqs.append(s)
        self._running_set_changed()
        return s

    def finish(self, seq: Sequence) -> None:
        """End a sequence: its pages and its state slot go back."""
        self.seqs.remove(seq)
        self._release(seq)
        self._running_set_changed()

    def _release(self, seq: Sequence) -> None:
        for blocks in self.span_blocks:
            blocks.release(seq)
            blocks.flush()
        if self.state_slots is not None:
            self.state_slots.release(seq)

    @torch.no_grad()
    def _forward_portions(self, portions, use_block_tables: bool = True):
        """Run portions [(sequence, first position, token ids)], at most one per
        sequence, through the model; hidden rows in the order of the tokens.  Metadata
        as in prepare_prefill (fastkernels/infra/engine.py:4902-4990): cu_seqlens,
        per-token slots and block tables, so attention reads the pages the store has
        just written.  In a chunked span a portion falls into one segment per chunk."""
        dev = self.device
        ids = np.concatenate([np.asarray(t, dtype=np.int64) for _, _, t in portions])
        pos = np.concatenate([np.arange(a, a + len(t), dtype=np.int64) for _, a, t in portions])
        i32 = []                           # all int32 metadata travels in one copy

        def put(a):
            a = np.ascontiguousarray(a, dtype=np.int32)
            i32.append(a.reshape(-1))
            return a.shape

        layout = []
        for blocks in self.span_blocks:
            segs, slots = [], []
            for s, a, t in portions:
                seg, sl = blocks.extend(s, a, len(t))
                segs += seg
                slots.append(sl)
            q = np.array([c for c, _, _ in segs])
            kv = np.array([k for _, k, _ in segs])
            bt = np.full((len(segs), max(len(pg) for _, _, pg in segs)), -1, dtype=np.int32)
            for j, (_, _, pg) in enumerate(segs):
                bt[j, :len(pg)] = pg
            layout.append((put(np.concatenate(slots)), put(bt), put(kv),
                           put(np.concatenate([[0], np.cumsum(q)])),
                           put(np.concatenate([[0], np.cumsum(kv)])), int(q.max()),
                           int(kv.max()), int(kv.sum())))
        state_shape = cu_shape = None
        if self.state_slots is not None:
            state_shape = put(np.repeat([s.state_slot for s, _, _ in portions],
                                        [len(t) for _, _, t in portions]))
            cu_shape = put(np.concatenate([[0], np.cumsum([len(t) for _, _, t in portions])]))
        flat = torch.from_numpy(np.concatenate(i32)).to(dev)
        at = 0

        def take(shape):
            nonlocal at
            n = int(np.prod(shape))
            v = flat[at:at + n].view(*shape)
            at += n
            return v

        spans = []
        for slots, bt, kv, cq, ck, *sizes in layout:
            spans.append(SpanBatch(take(slots), take(bt), take(kv), take(cq), take(ck), *sizes))
        first = spans[0]
        set_context(True, cu_seqlens_q=first.cu_seqlens_q, cu_seqlens_k=first.cu_seqlens_k,
                    max_seqlen_q=first.max_seqlen_q, max_seqlen_k=first.max_seqlen_k,
                    slot_mapping=first.slot_mapping,
                    block_tables=first.block_tables if use_block_tables else None, spans=spans,
                    state_slots=take(state_shape) if state_shape is not None else None,
                    cu_portions=take(cu_shape) if cu_shape is not None else None,
                    longest_portion=max(len(t) for _, _, t in portions))
        try:
            hidden = self.model(torch.from_numpy(ids).to(dev), torch.from_numpy(pos).to(dev))
        finally:
            reset_context()
        for blocks in self.span_blocks:
            blocks.flush()
        self._bt_dirty = True          # the page tables have grown
        self._ahead = None
        return hidden

    @torch.no_grad()
    def prefill(self, prompts, chunk_tokens: int | None = None,
                use_block_tables: bool = True) -> np.ndarray:
        """Run whole prompts through the model, fill their KV pages and sample the
        first new token of each (greedy); the sequences then join the running
        batch, ready for step().  Prefill side of ModelRunner.run
        (fastkernels/infra/engine.py:6048-6063).

        chunk_tokens=C splits the work into forwards of at most C tokens; a chunk
        attends over the pages written by earlier chunks plus itself (the
        reference's chunked prefill).  With a tensor-parallel communicator the
        chunk defaults to its row capacity.  use_block_tables=False (whole prompts
        of a model with one whole-context span only) attends over the batch's own
        dense K/V instead, the reference's path when no block table exists (its
        warm-up)."""
        from .comm import get_tp_comm
        comm = get_tp_comm()
        if chunk_tokens is None and comm is not None and comm.world > 1:
            chunk_tokens = comm.max_rows
        for prompt in prompts:
            n = len(prompt)
            if n < 1 or n + 1 > self.max_model_len:
                raise ValueError(f"prompt length {n} outside [1, {self.max_model_len - 1}]")
        if len(self.seqs) + len(prompts) > self.max_num_seqs:
            raise RuntimeError("max_num_seqs exceeded")
        new = [self._new_sequence(len(prompt)) for prompt in prompts]
        try:
            first = self._prefill_new(new, prompts, chunk_tokens, use_block_tables)
        except BaseException:
            for s in new:              # nothing joined: what they hold goes back
                self._release(s)
            raise
        for s, t in zip(new, first):
            s.num_tokens += 1          # the sampled token is the next step's input
            s.last_token = int(t)
            s.output.append(int(t))
            self.seqs.append(s)
        self._running_set_changed()
        return first

    def _prefill_new(self, new, prompts, chunk_tokens, use_block_tables) -> np.ndarray:
        done = [0] * len(new)
        first = np.zeros(len(new), dtype=np.int64)
        while any(d < len(pr) for d, pr in zip(done, prompts)):
            part = pack_prefill_chunk([len(pr) for pr in prompts], done, chunk_tokens)
            hidden = self._forward_portions(
                [(new[i], a, prompts[i][a:a + c]) for i, a, c in part],
                use_block_tables or chunk_tokens is not None)
            row_end = np.cumsum([c for _, _, c in part])
            ends = [(j, i) for j, (i, a, c) in enumerate(part) if a + c == len(prompts[i])]
            if ends:
                rows = torch.from_numpy(row_end[[j for j, _ in ends]].astype(np.int64) - 1)
                logits = self.model.project(hidden.index_select(0, rows.to(self.device)))
                vals, idxs = ops.argmax_rows(logits)
                tok = self.model.greedy(vals, idxs).cpu().numpy()
                for (j, i), t in zip(ends, tok):
                    first[i] = int(t)
            for i, a, c in part:
                done[i] = a + c
        return first

    @torch.no_grad()
    def feed(self, entries, want=None) -> list[torch.Tensor]:
        """Run the next tokens of open sequences, [(sequence, token ids)], and return
        for each entry the logits (fp32, on the host) at the places `want[i]` among its
        tokens (default: the last one).  Single tokens of sequences that already have
        some take the decode step, everything else goes through in portions; nothing
        is sampled.  Sequences fed here have no pending token: step() and feed() are
        not mixed on one sequence."""
        if want is None:
            want = [[len(t) - 1] for _, t in entries]
        if len({id(s) for s, _ in entries}) != len(entries):
            raise ValueError("at most one entry per sequence")
        for s, t in entries:
            if len(t) < 1 or s.num_tokens + len(t) > self.max_model_len:
                raise ValueError(f"sequence of {s.num_tokens} + {len(t)} tokens outside "
                                 f"[1, {self.max_model_len}]")
        single = [i for i, (s, t) in enumerate(entries) if len(t) == 1 and s.num_tokens > 0]
        rest = [i for i in range(len(entries)) if i not in set(single)]
        empty = torch.empty((0, self.model.logit_columns))
        out = [empty] * len(entries)
        if rest:
            hidden = self._forward_portions([(entries[i][0], entries[i][0].num_tokens,
                                              entries[i][1]) for i in rest])
            rows, o = [], 0
            for i in rest:
                rows += [o + int(w) for w in want[i]]
                o += len(entries[i][1])
                entries[i][0].num_tokens += len(entries[i][1])
            if rows:
                idx = torch.tensor(rows, dtype=torch.int64, device=self.device)
                logits = self.model.project(hidden.index_select(0, idx)).float().cpu()
                o = 0
                for i in rest:
                    out[i] = logits[o:o + len(want[i])]
                    o += len(want[i])
        if single:
            seqs = [entries[i][0] for i in single]
            for i in single:
                s, t = entries[i]
                s.num_tokens += 1
                s.last_token = int(t[0])
            self._ahead = None
            n = self.prepare_decode(True, seqs)
            bs = self.graph_batch_size(n)
            self.stage_inputs(n, bs, True)
            self.run_step_device(bs)
            self._mark_slot_in_flight()
            if any(len(want[i]) for i in single):
                logits = self.graph_vars["lm_logits"][:n].float().cpu()
                for j, i in enumerate(single):
                    out[i] = logits[j:j + 1].expand(len(want[i]), -1)
        return out

    def graph_batch_size(self, n: int) -> int:
        for bs in sorted(self.graphs):
            if bs >= n:
                return bs
        return n

    # ----------------------------------------------------------- host-side prep
    def prepare_decode(self, use_host_ids: bool, seqs=None) -> int:
        """Fill the pinned staging arrays for this step (engine.py:5793-5798) of the
        running sequences, or of `seqs`: position = n - 1 and, per span, context_len =
        keys visible from there and slot = place of the newest token in its pages.
        Everything but the token ids may already have been written while the previous
        step ran on the device (`_prepare_ahead`)."""
        if seqs is None and self._ahead is not None and \
                self._ahead == (self._seq_epoch, len(self.seqs)):
            n = len(self.seqs)
        else:
            n = self._prepare_layout(seqs)
        self._ahead = None
        if use_host_ids:
            ids = self.host_np["input_ids"]
            for i, s in enumerate(self.seqs if seqs is None else seqs):
                ids[i] = s.last_token
        return n

    def _prepare_ahead(self) -> None:
        """Called between the launch of a step and the wait for its tokens: the next
        step's positions, lengths, slots and block-table changes depend on no token
        value, so they are written into the next staging slot while the device is
        busy.  Skipped when the next step could fail (length limit, pool nearly
        empty), so that such errors are still raised by the step they belong to."""
        if not self.seqs or _NO_PREPARE_AHEAD:
            return
        if any(s.num_tokens > self.max_model_len for s in self.seqs):
            return
        for blocks in self.span_blocks:
            if sum(blocks.pages_missing(s) for s in self.seqs) > len(blocks.free):
                return
        self._prepare_layout()
        self._ahead = (self._seq_epoch, len(self.seqs))

    def _prepare_layout(self, seqs=None) -> int:
        seqs = self.seqs if seqs is None else seqs
        self._ring_pos = (self._ring_pos + 1) % self.RING
        ev = self._ring_events[self._ring_pos]
        if ev is not None:
            ev.synchronize()            # copies issued from this slot have landed
        self.host, self.host_np = self._ring[self._ring_pos], self._ring_np[self._ring_pos]
        h = self.host_np
        n = len(seqs)
        staged_for = tuple(s.seq_id for s in seqs)
        if staged_for != self._staged_for:
            self._bt_dirty = True
            self._staged_for = staged_for
        for i, s in enumerate(seqs):
            if s.num_tokens > self.max_model_len:
                raise RuntimeError("sequence exceeds max_model_len")
            pos = s.num_tokens - 1
            h["positions"][i] = pos
            for g, blocks in enumerate(self.span_blocks):
                if blocks.maybe_append_page(s):
                    self._bt_dirty = True
                h["span_lens"][g][i] = pos - blocks.base(pos) + 1
                h["span_slots"][g][i] = blocks.slot(s, pos)
            if self.state_slots is not None:
                h["state_slots"][i] = s.state_slot
        if self._bt_dirty:
            for g, bt in enumerate(h["span_tables"]):
                bt[:n].fill(-1)
                for i, s in enumerate(seqs):
                    bt[i, :len(s.table(g))] = s.table(g)
        return n

    def _mark_slot_in_flight(self) -> None:
        if self.device.type == "cuda":
            ev = self._ring_events[self._ring_pos]
            if ev is None:
                ev = self._ring_events[self._ring_pos] = torch.cuda.Event()
            ev.record()

    def stage_inputs(self, n: int, bs: int, use_host_ids: bool) -> None:
        """H2D copies from pinned memory into the graph's input buffers; padded
        rows get slot -1 / context_len 0 (engine.py:5404-5406)."""
        gv, h = self.graph_vars, self.host
        if bs > n:
            for slots, lens in zip(h["span_slots"], h["span_lens"]):
                slots[n:bs] = -1
                lens[n:bs] = 0
            if self.state_slots is not None:
                h["state_slots"][n:bs] = -1
            h["positions"][n:bs] = 0
        first = 0 if use_host_ids else 8 * self.max_num_seqs
        self._packed_dev[first:].copy_(h["packed"][first:], non_blocking=True)
        self.h2d_bytes += h["packed"].numel() - first
        if self._bt_dirty:
            for dst, src in zip(gv["span_tables"], h["span_tables"]):
                dst[:bs].copy_(src[:bs], non_blocking=True)
                self.h2d_bytes += src[:bs].numel() * 4
            self._bt_dirty = False

    # -------------------------------------------------------------- graph body
    def _forward(self, bs: int) -> None:
        gv = self.graph_vars
        self.model.begin_decode(get_context())
        hidden = self.model(gv["input_ids"][:bs], gv["positions"][:bs])
        gv["outputs"][:bs] = hidden
        logits = self.model.project(hidden)
        gv["lm_logits"][:bs] = logits
        ops.argmax_rows(gv["lm_logits"][:bs], gv["lm_max_vals"][:bs], gv["lm_max_idxs"][:bs])
        ids = self.model.greedy(gv["lm_max_vals"][:bs], gv["lm_max_idxs"][:bs])
        gv["token_ids"][:bs] = ids
        # hand the sampled ids to the next step on the device (engine.py:5689-5705)
        gv["input_ids"][:bs] = ids

    def _set_context(self, bs: int, max_ctx: int) -> None:
        gv = self.graph_vars
        cu = gv["cu_rows"][:bs + 1]
        spans = [SpanBatch(slots[:bs], tables[:bs], lens[:bs], cu)
                 for slots, lens, tables in zip(gv["span_slots"], gv["span_lens"],
                                                gv["span_tables"])]
        set_context(False, slot_mapping=gv["slot_mapping"][:bs],
                    context_lens=gv["context_lens"][:bs],
                    block_tables=gv["block_tables"][:bs], max_context_len=max_ctx, spans=spans,
                    state_slots=gv["state_slots"][:bs] if self.state_slots is not None else None,
                    cu_portions=cu if self.state_slots is not None else None)

    @torch.no_grad()
    def capture_cudagraph(self, batch_sizes) -> None:
        """Capture one graph per batch size with the persistent graph_vars as
        inputs; max_context_len is max_model_len at capture (engine.py:6832-6836)
        and the real lengths are read on the device at replay."""
        gv = self.graph_vars
        inputs = [self._packed_dev, *gv["span_tables"]]
        saved = [t.clone() for t in inputs]
        for slots, lens, tables in zip(gv["span_slots"], gv["span_lens"], gv["span_tables"]):
            slots.fill_(-1)
            lens.fill_(1)
            tables.fill_(0)
        if self.state_slots is not None:
            gv["state_slots"].fill_(-1)
        gv["positions"].zero_()
        gv["input_ids"].zero_()
        for bs in sorted(batch_sizes, reverse=True):
            self._set_context(bs, self.max_model_len)
            for _ in range(2):          # warm-up outside capture (lazy allocations, NCCL)
                self._forward(bs)
            torch.cuda.synchronize()
            graph = torch.cuda.CUDAGraph()
            with torch.cuda.graph(graph, self.graph_pool):
                self._forward(bs)
            if self.graph_pool is None:
                self.graph_pool = graph.pool()
            self.graphs[bs] = graph
            torch.cuda.synchronize()
            reset_context()
        for t, v in zip(inputs, saved):
            t.copy_(v)

    # -------------------------------------------------------------------- steps
    @torch.no_grad()
    def run_step_device(self, bs: int) -> None:
        """Replay (or eagerly run) the step for batch size `bs` on inputs that
        are already in the graph buffers."""
        g = self.graphs.get(bs)
        if g is not None and not self.enforce_eager:
            g.replay()
        else:
            self._set_context(bs, self.max_model_len)
            self._forward(bs)
            reset_context()

    @torch.no_grad()
    def step(self, sync: bool = True) -> np.ndarray | None:
        """One decode step for all running sequences through the public path:
        host prep -> pinned H2D staging -> graph replay -> D2H of the token ids.
        With sync=True the sampled ids come back to the host before returning
        and feed the next step from the host; with sync=False the next step
        reads them from the device buffer and the host copy is deferred."""
        n = self.prepare_decode(use_host_ids=sync)
        bs = self.graph_batch_size(n)
        self.stage_inputs(n, bs, use_host_ids=sync)
        self.run_step_device(bs)
        self.host["token_ids"][:n].copy_(self.graph_vars["token_ids"][:n], non_blocking=True)
        self._mark_slot_in_flight()
        self.d2h_bytes += n * 8
        for s in self.seqs:
            s.num_tokens += 1
        if not sync:
            return None
        landing = self.host_np["token_ids"]     # this step's slot (the next call moves on)
        self._prepare_ahead()
        torch.cuda.current_stream().synchronize()
        ids = landing[:n].copy()
        for s, t in zip(self.seqs, ids.tolist()):
            s.last_token = t
            s.output.append(t)
        return ids

    def device_status(self) -> int:
        """OR of every device status word this engine's kernels write (attention
        workspace word, the per-device default word of the row kernels and GEMMs,
        the tensor-parallel communicator's): 0 = no slot / page / position out of
        range and no wait ran out.  Synchronises; call between steps."""
        st = int(self.status.item()) | int(ops.default_status(self.device).item())
        if self.comm is not None:
            st |= int(self.comm.status.item())
        return st

    def decode(self, steps: int) -> np.ndarray:
        """Greedy-decode `steps` tokens for every running sequence; [steps, n].
        Raises if a kernel reported a device-side anomaly on the way."""
        toks = np.stack([self.step(sync=True) for _ in range(steps)])
        st = self.device_status()
        if st:
            if st & 4:
                # a wait ran out: a late stream-K contributor may have left its flag
                # raised, so the shared GEMM workspace starts the next call zeroed again
                ops.gemm_workspace(self.device)[:1024].zero_()
            raise RuntimeError(f"device status word {st} after decoding (fk_device_status bits)")
        return toks
