"""Mixture of experts: router, dispatch and grouped gated feed-forwards.

Every token has ``top`` routed slots and ``always`` more that name the same experts for every token (a shared expert as one
or several experts of the routed width: a gated feed-forward is the sum of the feed-forwards over blocks of its width).
Pairs (token, slot) are sorted by expert, so that an expert's tokens are consecutive rows; the weighted sum over a token's
slots happens where the result enters the residual stream (``Branch.pos`` / ``Branch.weight``).  With scored routing some
router outputs stand for the token's own row; their weights are summed per token (``Branch.self_weight``).

CUDA tensors run ``csrc/moe.cu`` and the grouped forms of the GEMM kernels; CPU tensors the plain-PyTorch statement.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn.functional as F

from . import GLU_ACTS, SM_COUNT, _p, _pdl, _s, effective_splits, gated_unit, native
from .latent import Branch

SMALL_TOKENS = 128      # up to here: one routing CTA, every expert's GEMM reads the step's own rows, no gather
CHUNK_TOKENS = 64       # tokens per routing CTA above
TILE_ROWS = 128         # rows of a grouped prefill tile
TILE_ROWS_F32 = 64


@dataclass
class Routing:
    """``pos [T, K]``: row of each pair in expert order (-1: the token takes no part); ``weight [T, K]``; ``row_token [T * K]``:
    the token of each row; ``groups [n, 4]``: (expert, first row, rows, 0) per tile of at most ``tile_rows`` rows, the first
    ``n_groups[0]`` of them in use."""

    pos: torch.Tensor
    weight: torch.Tensor
    row_token: torch.Tensor
    groups: torch.Tensor
    n_groups: torch.Tensor
    tile_rows: int
    self_weight: Optional[torch.Tensor] = None   # [T] weight of the token's own row (scored routing)


@dataclass(frozen=True)
class Scored:
    """Routing by scores: softmax over all ``experts + identity`` outputs; ``correction`` (fp32, one per output) enters the choice
    only, which is among the ``keep`` best of ``groups`` equal runs of outputs (a group is as good as its best output); the
    weights are the chosen scores over their sum, times ``scale``.  ``always_gate``: one more logit, behind the others, whose
    sigmoid weighs the always-on experts.  ``sigmoid``: the scores are the outputs' sigmoids, not divided by their sum;
    ``group_best`` 2: a group is as good as the sum of its two best outputs."""

    correction: torch.Tensor
    identity: int = 0
    groups: int = 1
    keep: int = 1
    scale: float = 1.0
    always_gate: bool = False
    sigmoid: bool = False
    group_best: int = 1


def _max_groups(T: int, top: int, experts: int, always: int, tile_rows: int) -> int:
    """Most tiles the pairs of ``T`` tokens can make: every expert in use ends in a partial one."""
    if tile_rows >= T:
        return min(experts, T * top) + always
    return min(experts, T * top) + T * top // tile_rows + always * (1 + T // tile_rows)


def _choose_cpu(z: torch.Tensor, top: int, experts: int, s: Scored):
    """(expert [T, top], ``experts`` where it is the token's own row; weight [T, top]; weight of the own row [T])"""
    n = experts + s.identity
    score = torch.sigmoid(z[:, :n]) if s.sigmoid else torch.softmax(z[:, :n], 1)
    choice = score + s.correction
    size = n // s.groups
    best = choice.view(-1, s.groups, size).topk(min(s.group_best, size), 2).values.sum(2).sort(dim=1, descending=True, stable=True).indices[:, :s.keep]
    open_ = torch.zeros(z.shape[0], s.groups, dtype=torch.bool).scatter_(1, best, True).repeat_interleave(size, 1)
    chosen = choice.masked_fill(~open_, float("-inf")).sort(dim=1, descending=True, stable=True).indices[:, :top]
    w = score.gather(1, chosen)
    w = (w if s.sigmoid else w / (w.sum(1, keepdim=True) + 1e-20)) * s.scale
    own = chosen >= experts
    return chosen.clamp_max(experts), w.masked_fill(own, 0.0), (w * own).sum(1)


def route(logits: Branch, top: int, experts: int, always: int, slots: torch.Tensor, *, f32: bool = False,
          scored: Optional[Scored] = None) -> Routing:
    """The ``top`` largest of the fp32 router logits ``[T, experts]`` per token (lowest expert first among equals), softmax over
    those alone, or as ``scored`` says; then slots for experts ``experts .. experts + always - 1`` of weight one.  Tokens whose
    cache slot is negative (padding rows of a decode graph) take no part."""
    src = logits.slabs if logits.slabs is not None else logits.rows
    T, dev = src.shape[-2], src.device
    K, E = top + always, experts + always
    small = T <= SMALL_TOKENS
    if not src.is_cuda:
        z = logits.value()
        own, always_w = None, torch.ones(T, 1)
        if scored is not None:
            expert, weight, own = _choose_cpu(z, top, experts, scored)
            expert = torch.where(expert < experts, expert, E)
            if scored.always_gate:
                always_w = torch.sigmoid(z[:, experts + scored.identity:experts + scored.identity + 1])
        else:
            order = torch.sort(z[:, :experts], dim=1, descending=True, stable=True)
            expert, weight = order.indices[:, :top], torch.softmax(order.values[:, :top], 1)
        expert = torch.cat([expert, torch.arange(experts, E).expand(T, always)], 1)
        weight = torch.cat([weight, always_w.expand(T, always)], 1)
        live = (slots >= 0)[:, None].expand(T, K)
        expert = torch.where(live, expert, E)
        by_expert = torch.sort(expert.reshape(-1), stable=True).indices
        n = int((expert < E).sum())
        pos = torch.full((T * K,), -1, dtype=torch.int32)
        pos[by_expert[:n]] = torch.arange(n, dtype=torch.int32)
        counts = torch.bincount(expert.reshape(-1), minlength=E + 1)[:E].tolist()
        groups, first = [], 0
        for e, c in enumerate(counts):
            if c:
                groups.append((e, first, c, 0))
            first += c
        return Routing(pos.view(T, K), torch.where(live, weight, torch.zeros(())), (by_expert // K).int(),
                       torch.tensor(groups, dtype=torch.int32).view(-1, 4), torch.tensor([len(groups)], dtype=torch.int32), max(1, T),
                       None if own is None else torch.where(slots >= 0, own, torch.zeros(())))
    s = logits.slabs
    assert s is not None and s.dtype == torch.float32 and s.stride(2) == 1 and slots.dtype == torch.int64
    tile = TILE_ROWS_F32 if f32 else (T if small else TILE_ROWS)
    chunk = SMALL_TOKENS if small else CHUNK_TOKENS
    chunks = -(-T // chunk)
    i32 = dict(dtype=torch.int32, device=dev)
    pos, row_token = torch.empty((T, K), **i32), torch.empty((T * K,), **i32)
    weight = torch.empty((T, K), dtype=torch.float32, device=dev)
    expert = torch.empty((T, K), **i32)
    counts = torch.empty((chunks, E), **i32)
    groups = torch.empty((_max_groups(T, top, experts, always, tile), 4), **i32)
    n_groups = torch.empty((1,), **i32)
    args = (_p(expert), _p(pos), _p(weight), _p(row_token), _p(counts), _p(groups), groups.shape[0], _p(n_groups), T, top, experts, always,
            chunk, tile)
    own, rule = None, (None, None, experts, 1, 1, -1, 1.0, 0, 1)
    if scored is not None:
        n = experts + scored.identity
        assert scored.correction.dtype == torch.float32 and scored.correction.shape == (n,) and s.shape[2] >= n + scored.always_gate
        own = torch.empty((T,), dtype=torch.float32, device=dev)
        rule = (_p(scored.correction), _p(own), n, scored.groups, scored.keep, n if scored.always_gate else -1, float(scored.scale),
                1 if scored.sigmoid else 0, scored.group_best)
    native.call("prism_moe_route", _p(s), s.stride(0), s.stride(1), s.shape[0], _p(slots), *args, *rule, _s(), _pdl())
    if chunks > 1:
        native.call("prism_moe_place", *args, _s(), _pdl())
    return Routing(pos, weight, row_token, groups, n_groups, tile, own)


def _down_splits(m: int, k: int, groups: int) -> int:
    kb = -(-k // 64)
    return max(1, min(SM_COUNT // max(1, groups * -(-m // 128)), kb // 4 if kb >= 8 else 1, 8))


def expert_ffn(x: torch.Tensor, r: Routing, w_gate_up: torch.Tensor, w_down: torch.Tensor, act: str = "silu",
               limit: float = 0.0) -> Branch:
    """Every pair's ``down_e(act(gate_e x) * up_e x)`` as a branch whose value is the weighted sum per token.  ``w_gate_up``
    ``[E, 2 F, W]`` (gate rows, then up rows), ``w_down [E, W, F]``; ``act`` as in ``gated_unit``, with its ``limit``."""
    T, W = x.shape
    E, F2, _ = w_gate_up.shape
    I = F2 // 2
    K = r.pos.shape[1]
    N = T * K
    if not x.is_cuda:
        y = torch.zeros((N, W))
        for e, first, count, _ in r.groups.tolist():
            h = x[r.row_token[first:first + count].long()].float() @ w_gate_up[e].float().t()
            a = gated_unit(h[:, :I], h[:, I:], act, limit).to(x.dtype).float()
            y[first:first + count] = a @ w_down[e].float().t()
        return Branch(slabs=y.unsqueeze(0), pos=r.pos, weight=r.weight, self_weight=r.self_weight)
    assert x.dtype == w_gate_up.dtype == w_down.dtype and x.stride(1) == 1 and w_gate_up.is_contiguous() and w_down.is_contiguous()
    dev, G = x.device, r.groups.shape[0]
    table = (_p(r.groups), G, _p(r.n_groups))
    if x.dtype == torch.float32:
        gu = torch.empty((N, F2), dtype=torch.float32, device=dev)
        native.call("prism_gemm_f32_grouped", _p(w_gate_up), _p(x), _p(gu), F2, N, W, W, x.stride(0), F2, *table, _p(r.row_token), T, E, _s(),
                    _pdl())
        a = torch.empty((N, I), dtype=torch.float32, device=dev)
        native.call("prism_glu_f32", _p(gu), _p(a), N, I, GLU_ACTS[act], float(limit), _s(), _pdl())
        y = torch.empty((1, N, W), dtype=torch.float32, device=dev)
        native.call("prism_gemm_f32_grouped", _p(w_down), _p(a), _p(y), W, N, I, I, I, W, *table, None, N, E, _s(), _pdl())
        return Branch(slabs=y, pos=r.pos, weight=r.weight, self_weight=r.self_weight)
    a = torch.empty((N, I), dtype=torch.bfloat16, device=dev)
    if T <= SMALL_TOKENS:
        native.call("prism_gemm_grouped_small", _p(w_gate_up), _p(x), _p(a), I, T, T, W, x.stride(0), I, *table, _p(r.row_token), N, E,
                    GLU_ACTS[act], float(limit), 1, 0, _s(), _pdl())
        splits = effective_splits(I, _down_splits(W, I, G))
        y = torch.empty((splits, N, W), dtype=torch.float32, device=dev)
        native.call("prism_gemm_grouped_small", _p(w_down), _p(a), _p(y), W, T, N, I, I, W, *table, None, N, E, 0, 0.0, splits, y.stride(0), _s(),
                    _pdl())
        return Branch(slabs=y, pos=r.pos, weight=r.weight, self_weight=r.self_weight)
    rows = torch.empty((N, W), dtype=torch.bfloat16, device=dev)
    native.call("prism_moe_gather", _p(x), x.stride(0), _p(r.pos), _p(rows), T, K, W, _s(), _pdl())
    native.call("prism_gemm_grouped", _p(w_gate_up), _p(rows), _p(a), I, N, W, W, I, *table, E, GLU_ACTS[act], float(limit), _s(), _pdl())
    y = torch.empty((N, W), dtype=torch.bfloat16, device=dev)
    native.call("prism_gemm_grouped", _p(w_down), _p(a), _p(y), W, N, I, I, W, *table, E, 0, 0.0, _s(), _pdl())
    return Branch(rows=y, pos=r.pos, weight=r.weight, self_weight=r.self_weight)
