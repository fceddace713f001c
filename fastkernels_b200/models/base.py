"""What the engine asks of a model.

A served model is an nn.Module whose forward(input_ids, positions) returns one
hidden row per token; the step's batch metadata comes from
fastkernels_b200.infra.context.get_context().
"""
from __future__ import annotations


class ServedModel:
    # True: the model keeps recurrent state and reads ctx.state_slots / cu_portions
    uses_state: bool = False

    @classmethod
    def spans_of(cls, config) -> list:
        """One entry per span of the attention layers: chunk size in tokens, None =
        the whole context (see fastkernels_b200.cache)."""
        return [None]

    @property
    def kv_spans(self) -> list:
        return self.spans_of(self.config)

    def init_random(self, seed: int, scale: float, rank: int = 0) -> None:
        """Random weights of the configured architecture."""
        raise NotImplementedError

    def load_tensors(self, source) -> None:
        """Weights from a models.weights.TensorSource."""
        raise NotImplementedError

    def allocate_kv(self, num_blocks: list[int], block_size: int, device):
        """Allocate the page pools (pages per span) and hand them to the layers."""
        raise NotImplementedError

    def allocate_state(self, num_slots: int, device) -> None:
        """Allocate recurrent state for `num_slots` sequences."""

    def preallocate(self, max_num_seqs: int, max_model_len: int, device, max_splits: int):
        """Workspaces that must not move between graph replays; returns the device
        status word of the model's kernels."""
        raise NotImplementedError

    def begin_decode(self, ctx) -> None:
        """Once per decode step, before forward: schedules that all layers share."""

    def project(self, hidden):
        """Logits of hidden rows."""
        raise NotImplementedError

    def greedy(self, max_vals, max_idxs):
        """Token ids from the per-row (max, index) pairs of this rank's logits."""
        return max_idxs

    @property
    def hidden_columns(self) -> int:
        """Columns of a hidden row."""
        raise NotImplementedError

    @property
    def logit_columns(self) -> int:
        """Columns of a logit row on this rank."""
        raise NotImplementedError
