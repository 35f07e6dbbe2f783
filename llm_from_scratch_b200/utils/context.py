"""Process-global attention metadata handed from the model runner to the attention layers.

Same fields and accessors as the reference's utils/context.py:5-27, so a model written against the
reference's context reads this one unchanged.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

import torch


@dataclass
class Context:
    is_prefill: bool = False
    cu_seqlens_q: Optional[torch.Tensor] = None   # int32 [num_seqs + 1]
    cu_seqlens_k: Optional[torch.Tensor] = None   # int32 [num_seqs + 1]
    max_seqlen_q: int = 0
    max_seqlen_k: int = 0
    slot_mapping: Optional[torch.Tensor] = None   # int64 [num_tokens], -1 = skip
    context_lens: Optional[torch.Tensor] = None   # int64 [batch] (decode)
    block_tables: Optional[torch.Tensor] = None   # int32 [batch, max_blocks], -1 padded
    # not in the reference (its runner builds no positions although the model needs them for RoPE):
    positions: Optional[torch.Tensor] = None      # int64 [num_tokens]; None in decode = context_lens - 1
    prefill_plan: object = None                   # ops.PrefillPlan of this step's cu_seqlens_q, or None
    state_slots: Optional[torch.Tensor] = None    # int64 [num_seqs] slot of every sequence's recurrent state, -1 = none
    logit_rows: Optional[torch.Tensor] = None     # int64 rows whose logits are wanted; None = each sequence's last
    singles: Optional["Singles"] = None           # the step in its two parts, for models that serve them apart
    portions: Optional["Portions"] = None


@dataclass
class Singles:
    """The leading sequences of a step that bring one token each: row i of the step belongs to sequence i."""
    rows: int
    context_lens: torch.Tensor                    # int64 [rows], the new token included
    block_tables: torch.Tensor                    # int32 [rows, max_blocks]
    state_slots: Optional[torch.Tensor]           # int64 [rows]


@dataclass
class KeyRange:
    """The keys that the portions of a step reach: the ends of their contexts, packed."""
    cu_seqlens_k: torch.Tensor                    # int32 [n + 1], starts at 0
    max_seqlen_k: int
    total_k: int
    has_prefix: bool                              # some of them came in an earlier step


@dataclass
class Portions:
    """The other sequences of a mixed step: prompts and portions of prompts, ragged, behind the singles' rows."""
    num_tokens: int                               # rows of the step that belong to a sequence, singles included (a bound
                                                  # in captured steps)
    cu_seqlens_q: torch.Tensor                    # int32 [n + 1], rows of the step
    cu_seqlens_k: torch.Tensor                    # int32 [n + 1], starts at 0
    max_seqlen_q: int
    max_seqlen_k: int
    total_k: int                                  # tokens of all contexts
    has_prefix: bool                              # some context is longer than its portion
    block_tables: torch.Tensor                    # int32 [n, max_blocks]
    state_slots: Optional[torch.Tensor]           # int64 [n]
    captured: bool = False                        # part of a CUDA graph: lengths differ from replay to replay
    ranges: dict = field(default_factory=dict)    # window -> KeyRange, for the windows the model's layers have
    chunk_ranges: dict = field(default_factory=dict)   # the same by chunk size, for layers that attend inside chunks
    plans: dict = field(default_factory=dict)     # tile lists by rows per tile, built when a layer asks

    def keys(self, window: int = 0, chunk: int = 0) -> KeyRange:
        """What a layer with this sliding window, or with chunks of this size, needs of the contexts (0: all of them)."""
        if chunk in self.chunk_ranges:
            return self.chunk_ranges[chunk]
        if window in self.ranges:
            return self.ranges[window]
        return KeyRange(self.cu_seqlens_k, self.max_seqlen_k, self.total_k, self.has_prefix)

    def plan(self, tile_rows: int):
        if tile_rows <= 0:
            return None
        if tile_rows not in self.plans:
            from .. import ops
            self.plans[tile_rows] = ops.prefill_plan(self.cu_seqlens_q, self.num_tokens, self.max_seqlen_q, tile_rows)
        return self.plans[tile_rows]


_current = Context()


def get_context() -> Context:
    return _current


def set_context(is_prefill, cu_seqlens_q=None, cu_seqlens_k=None, max_seqlen_q=0, max_seqlen_k=0,
                slot_mapping=None, context_lens=None, block_tables=None, positions=None,
                prefill_plan=None, state_slots=None, logit_rows=None, singles=None, portions=None) -> None:
    global _current
    _current = Context(is_prefill, cu_seqlens_q, cu_seqlens_k, max_seqlen_q, max_seqlen_k,
                       slot_mapping, context_lens, block_tables, positions, prefill_plan,
                       state_slots, logit_rows, singles, portions)


def reset_context() -> None:
    global _current
    _current = Context()
