"""Replay of given token ids through an engine, step by step, for their logits.

A ``TraceReplay`` drives the engine's own block manager, input preparation and model runner: a step is one
batch of (request, next tokens) entries, portions of prompts beside single tokens, computed from the pages that
earlier steps filled.  Nothing is sampled, and the scheduler does not choose the batches: the trace does.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Hashable, Iterable, Sequence as Seq

import torch

from .contracts import BatchPlan, Phase, PrefillSlice
from .request import RequestState
from .sequence import Sequence


@dataclass(frozen=True)
class ReplayEntry:
    request: Hashable
    tokens: Seq[int]
    want: Seq[int] = ()        # places among ``tokens`` whose logits are asked for


class TraceReplay:
    def __init__(self, engine) -> None:
        self.engine = engine
        self.blocks = engine.scheduler.block_manager
        if engine.config.enable_prefix_caching:
            raise ValueError("a replay computes every token it is given: build the engine with enable_prefix_caching=False")
        self._live: dict[Hashable, Sequence] = {}

    def _advance(self, entry: ReplayEntry) -> tuple[Sequence, PrefillSlice]:
        """Admit the request or append its tokens; pages for everything it now holds."""
        tokens = [int(t) for t in entry.tokens]
        if not tokens:
            raise ValueError(f"request {entry.request!r}: a step entry needs at least one token")
        vocab = self.engine.arch.vocab_size
        if min(tokens) < 0 or max(tokens) >= vocab:
            raise ValueError(f"request {entry.request!r}: token id outside the vocabulary of {vocab}")
        seq = self._live.get(entry.request)
        if seq is None:
            seq = Sequence(self.engine._ids(), tokens, image_token_id=self.engine.arch.image_token_id,
                           video_token_id=self.engine.arch.video_token_id)
            start = 0
            self.blocks.allocate(seq)
            seq.lifecycle.transition(RequestState.PREFILLING, "replay")
            self._live[entry.request] = seq
        else:
            start = len(seq)
            for t in tokens:
                seq.append_token(t)
            self.blocks.grow(seq)
        if len(seq) > self.engine.config.max_model_len:
            raise ValueError(f"request {entry.request!r}: {len(seq)} tokens exceed max_model_len {self.engine.config.max_model_len}")
        return seq, PrefillSlice(start, len(tokens))

    def step(self, entries: Iterable[ReplayEntry], end: Iterable[Hashable] = ()) -> torch.Tensor:
        """Run one batch; fp32 logits ``[wanted, vocab]`` (CPU) in the order of the entries and of their ``want``.
        The requests in ``end`` give their pages back afterwards."""
        entries = list(entries)
        logits = torch.empty((0, self.engine.arch.vocab_size), dtype=torch.float32)
        if entries:
            if len({e.request for e in entries}) != len(entries):
                raise ValueError("a request appears twice in one step")
            pairs = [self._advance(e) for e in entries]
            seqs, slices = tuple(s for s, _ in pairs), tuple(sl for _, sl in pairs)
            rows, base = [], 0
            for e, sl in zip(entries, slices):
                if any(not 0 <= int(w) < sl.length for w in e.want):
                    raise ValueError(f"request {e.request!r}: wanted place outside its {sl.length} tokens")
                rows += [base + int(w) for w in e.want]
                base += sl.length
            decode = all(sl.length == 1 and sl.start > 0 for sl in slices)
            plan = (BatchPlan(Phase.DECODE, seqs, (), num_tokens=base) if decode
                    else BatchPlan(Phase.PREFILL, seqs, slices, num_tokens=base))
            logits = self.engine.executor.step_logits(plan, rows)
            for s, sl in pairs:
                s.num_computed_tokens = sl.end
        for request in end:
            self.blocks.deallocate(self._live.pop(request))
        return logits
