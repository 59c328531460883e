"""What every model family shares with the runner: the attention metadata of a step and the collective hooks
of a tensor-parallel rank."""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

import torch

from .. import ops

# at or below this many tokens the GEMMs are weight-streaming: split-K + fp32 partials
SMALL_T = 128


@dataclass
class AttnMeta:
    """Device-side attention metadata of one step."""

    is_prefill: bool
    block_tables: torch.Tensor                     # [S, max_blocks] int32
    slots: torch.Tensor                            # [T] int64 flat KV slots of the new tokens
    # prefill
    cu_seqlens_q: Optional[torch.Tensor] = None    # [S+1] int32
    kv_lens: Optional[torch.Tensor] = None         # [S] int32 keys visible (history + chunk)
    cu_seqlens_kv: Optional[torch.Tensor] = None   # [S+1] int32 running sum of kv_lens (None: the page-reading kernel)
    total_kv: int = 0                              # sum and maximum of kv_lens, known on the host
    max_kv_len: int = 0
    max_q_len: int = 0
    last_rows: Optional[torch.Tensor] = None       # [S] int64 row of each sequence's last token
    no_history: bool = False                       # every sequence attends only to this chunk's own keys
    # decode
    context_lens: Optional[torch.Tensor] = None    # [B] int32 (including the new token)
    nsplit: int = 0
    workspace: Optional[tuple[torch.Tensor, torch.Tensor]] = None
    # prefill with the attention pruning strategy: collects last-query attention over visual tokens
    scorer: Optional[object] = None
    # recurrent layers: the state container and the slot of each sequence (decode: of each row, < 0: padding)
    state: Optional[object] = None                 # ops.recurrent.StateCache
    state_slots: Optional[torch.Tensor] = None     # [S] int32
    host_lens: Optional[list] = None               # (new tokens, tokens up to the last of them) per sequence, on the host
    plans: dict = field(default_factory=dict)      # what a step's layers derive from them once
    attended_pairs: int = 0                        # sum over the sequences of query rows x visible keys, known on the host


class TPComm:
    """Collective hooks of a tensor-parallel rank; the single-rank default does nothing."""

    rank = 0
    size = 1

    def reduce_partials(self, partials: torch.Tensor) -> torch.Tensor:
        """fp32 ``[S, T, H]`` rank-local partial slabs -> slabs whose sum is the full result."""
        return partials

    def reduce_dense(self, x: torch.Tensor) -> torch.Tensor:
        """bf16 ``[T, H]`` rank-local partial result -> summed over ranks."""
        return x

    def greedy_merge(self, local_val: torch.Tensor, local_id: torch.Tensor) -> torch.Tensor:
        return local_id

    def gather_logits(self, logits: torch.Tensor) -> torch.Tensor:
        return logits

    def all_gather_rows(self, x: torch.Tensor) -> torch.Tensor:
        return x

    def begin_step(self) -> None:
        return None

    def row_parallel(self, x: torch.Tensor, w: torch.Tensor, stages: int = 0):
        """Row-parallel projection -> ``(dense, partials, ticket)``; exactly one is set.
        ``stages`` caps the operand ring of a decode-sized launch (0 = as deep as fits)."""
        T = x.shape[0]
        # short prefills (up to 511 tokens) split K too: o_proj and down_proj have 32 weight tiles at 8B widths,
        # one CTA each would leave 116 SMs idle
        if T <= SMALL_T or (x.is_cuda and T <= ops.SPLIT_K_MAX_TOKENS):
            splits = ops.choose_splits(w.shape[0], w.shape[1], T) if x.is_cuda else 1
            if splits > 1 or T <= SMALL_T:
                return None, ops.linear_partial(x, w, splits, stages=stages), None
        return ops.linear(x, w), None, None

    def add_rmsnorm(self, weight, eps, dense, partials, ticket, residual, extra=None, extra_index=None):
        """``(normed, new_residual)`` from whatever ``row_parallel`` returned."""
        return ops.add_rmsnorm(weight, eps, x=dense, partials=partials, residual=residual, extra=extra,
                               extra_index=extra_index)
