"""Host-side cache management: running sequences, KV pages and recurrent-state slots.

A model's attention layers fall into SPANS.  A span says which part of a sequence
its layers can see: the whole context (chunk None), or only the current chunk of
`chunk` tokens, counted from position 0.  Every span has its own page pool and its
own page table per sequence.  Pages of a chunked span hold ONE chunk: position p
sits at offset p % chunk of the chunk's own pages, so inside the chunk attention is
ordinary causal attention over an ordinary page table, and a finished chunk's pages
go back to the pool.

BlockManager is the page side of fastkernels/infra/engine.py:380-586 (decode
subset) with the chunked span added.
"""
from __future__ import annotations

from dataclasses import dataclass, field

import numpy as np


@dataclass
class Sequence:
    """One running request: `num_tokens` counts the tokens whose K/V are (or, for
    the newest one, are about to be) in the cache; `tables[g]` lists its pages in
    span g, which start at position `bases[g]`; `state_slot` is its recurrent-state
    slot (-1: the model keeps none)."""
    seq_id: int
    num_tokens: int
    last_token: int = 0
    output: list[int] = field(default_factory=list)
    tables: dict = field(default_factory=dict)
    bases: dict = field(default_factory=dict)
    state_slot: int = -1

    def table(self, span: int) -> list[int]:
        return self.tables.setdefault(span, [])

    @property
    def block_table(self) -> list[int]:
        return self.table(0)


class BlockManager:
    """Free-list page allocator of one span."""

    def __init__(self, num_blocks: int, block_size: int, span: int = 0,
                 chunk: int | None = None):
        self.block_size = block_size
        self.span = span
        self.chunk = chunk
        self.num_blocks = num_blocks
        self.free = list(range(num_blocks - 1, -1, -1))
        self._retired: list[int] = []

    def max_blocks(self, max_len: int) -> int:
        """Page-table columns a sequence of up to max_len tokens needs."""
        longest = max_len if self.chunk is None else min(max_len, self.chunk)
        return (longest + self.block_size - 1) // self.block_size

    def base(self, pos: int) -> int:
        """First position that a query at `pos` can see."""
        return 0 if self.chunk is None else pos // self.chunk * self.chunk

    def _grow(self, seq: Sequence, pos: int) -> bool:
        """Make sure the page of position `pos` exists; True if the table changed."""
        changed = False
        table, base = seq.table(self.span), self.base(pos)
        if seq.bases.get(self.span, 0) != base:
            self._retired.extend(reversed(table))
            table.clear()
            changed = True
        seq.bases[self.span] = base
        need = (pos - base) // self.block_size + 1
        while len(table) < need:
            table.append(self._pop())
            changed = True
        return changed

    def slot(self, seq: Sequence, pos: int) -> int:
        off = pos - self.base(pos)
        return seq.table(self.span)[off // self.block_size] * self.block_size \
            + off % self.block_size

    def allocate(self, seq: Sequence) -> None:
        """Pages for all of the sequence's tokens that a next one can still see."""
        self._grow(seq, seq.num_tokens - 1)
        self.flush()

    def maybe_append_page(self, seq: Sequence) -> bool:
        """Called with num_tokens INCLUDING the token sampled last step: a new
        page is needed when that token is the first of a page (engine.py:530-533)."""
        changed = self._grow(seq, seq.num_tokens - 1)
        self.flush()
        return changed

    def pages_missing(self, seq: Sequence) -> int:
        """Pages that maybe_append_page would take from the pool."""
        pos = seq.num_tokens - 1
        have = len(seq.table(self.span)) if seq.bases.get(self.span, 0) == self.base(pos) else 0
        return max(0, (pos - self.base(pos)) // self.block_size + 1 - have)

    def extend(self, seq: Sequence, start: int, count: int):
        """Pages for tokens start .. start + count - 1.  Returns (segments, slots): one
        segment (number of queries, number of keys up to the last of them, pages) per
        chunk the tokens touch, and the cache slot of every token.  Pages of chunks
        finished on the way stay reserved until flush()."""
        segments, slots = [], []
        a, end = start, start + count
        while a < end:
            base = self.base(a)
            b = end if self.chunk is None else min(end, base + self.chunk)
            self._grow(seq, a)
            self._grow(seq, b - 1)
            pages = np.asarray(seq.table(self.span), dtype=np.int64)
            off = np.arange(a - base, b - base)
            slots.append(pages[off // self.block_size] * self.block_size
                         + off % self.block_size)
            segments.append((b - a, b - base, pages))
            a = b
        return segments, np.concatenate(slots).astype(np.int32)

    def flush(self) -> None:
        """Give back the pages of finished chunks: nothing launched from here on
        reads them before it has written them."""
        self.free.extend(self._retired)
        self._retired.clear()

    def _pop(self) -> int:
        if not self.free:
            raise RuntimeError("KV pool exhausted")
        return self.free.pop()

    def release(self, seq: Sequence) -> None:
        self.free.extend(reversed(seq.table(self.span)))
        seq.table(self.span).clear()
        seq.bases.pop(self.span, None)


class StateSlots:
    """Slots of recurrent state, one per running sequence.  A slot needs no clearing:
    the kernels start from zero at position 0."""

    def __init__(self, num_slots: int):
        self.num_slots = num_slots
        self.free = list(range(num_slots - 1, -1, -1))

    def allocate(self, seq: Sequence) -> None:
        if seq.state_slot < 0:
            if not self.free:
                raise RuntimeError("recurrent-state slots exhausted")
            seq.state_slot = self.free.pop()

    def release(self, seq: Sequence) -> None:
        if seq.state_slot >= 0:
            self.free.append(seq.state_slot)
            seq.state_slot = -1


def pack_prefill_chunk(prompt_lens, done, budget):
    """Next prefill forward: walk the sequences in order and take as many of each
    one's remaining prompt tokens as the token budget allows (None = no limit).
    Returns [(sequence index, first token, count)]; every sequence appears at most
    once, so a forward holds at most one chunk per sequence."""
    left = budget if budget is not None else 1 << 62
    part = []
    for i, n in enumerate(prompt_lens):
        take = min(n - done[i], left)
        if take > 0:
            part.append((i, done[i], take))
            left -= take
        if left == 0:
            break
    return part
