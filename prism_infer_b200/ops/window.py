"""Windowed grouped-query attention over single-row paged caches, plain or differential, and the token-side gate.

A token's cache row holds all heads' keys and values of a layer: ``[key heads x maps x dq | value heads x dv]``.  A query at
position ``i`` sees key ``j`` when ``j <= i`` and (``i - j < window`` or ``j < keep_first``).  With two maps every head has two
queries and two keys over one value; the second map's output is subtracted ``lam`` times and the difference normalised.  Scores
may be bounded (``softcap``), a sink per head may join the softmax's denominator, the values may be the keys as projected, and
a layer may attend with its queries alone over another layer's cache rows.

CUDA tensors run the kernels of ``csrc/window_attention.cu`` (bf16, or true 32-bit on fp32 tensors) and raise without them;
CPU tensors run the plain-PyTorch statement.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn.functional as F

from . import SM_COUNT, KVCache, _decode_counters, _p, _pdl, _s, native
from .latent import Branch

TC_MAX_HEAD = 128        # widest key map and value head of the tcgen05 prefill kernel
TC_MAX_KEY = 192         # widest key head with a single map
MMA_MAX_KEY = 512        # widest key row (all maps) and value head of the mma.sync decode kernel
MMA_MAX_VALUE = 256
MAX_SPLITS = 32
KEY_TILE = 64


@dataclass(frozen=True)
class WindowSpec:
    """Sizes and constants of one mixer.  ``dq`` and ``dv`` are ``dim`` and ``vdim`` padded to multiples of 16 with zeros."""

    heads: int
    kv_heads: int
    maps: int
    dim: int
    vdim: int
    rot_dims: int
    scale: float
    window: int
    keep_first: int
    gate: bool
    eps: float
    lam: float = 0.0         # weight of the second map
    gain: float = 1.0        # factor on the normalised difference
    head_norm: bool = False  # norm weights of one head, for every head
    tied: bool = False       # the values are the keys before norm and rotation: no rows of their own in the projection
    shared: bool = False     # queries only: keys and values are another layer's
    softcap: float = 0.0     # scores become softcap * tanh(score / softcap); 0: as they are

    @property
    def dq(self) -> int:
        return -(-self.dim // 16) * 16

    @property
    def dv(self) -> int:
        return -(-self.vdim // 16) * 16

    @property
    def q_cols(self) -> int:
        return self.heads * self.maps * self.dq

    @property
    def k_cols(self) -> int:
        return self.kv_heads * self.maps * self.dq

    @property
    def v_cols(self) -> int:
        return self.kv_heads * self.dv

    @property
    def gate_row(self) -> int:
        """First gate row of the stacked projection."""
        return self.q_cols + (0 if self.shared else self.k_cols + (0 if self.tied else self.v_cols))

    @property
    def proj_cols(self) -> int:
        """Rows of the stacked projection: queries, keys, values (those it has) and (padded to 16) one gate per head."""
        return self.gate_row + (-(-self.heads // 16) * 16 if self.gate else 0)


@dataclass
class WindowWeights:
    """What the projection's outputs meet on their way to the cache: bias over all stacked rows, norm weights over the whole
    query and key rows or over a head, rotary frequencies (fp32); each may be absent.  ``sink [H]`` (fp32): scores that take
    part in the softmax's denominator only."""

    bias: Optional[torch.Tensor] = None
    q_norm: Optional[torch.Tensor] = None
    k_norm: Optional[torch.Tensor] = None
    inv_freq: Optional[torch.Tensor] = None
    sink: Optional[torch.Tensor] = None


def _rotate(x: torch.Tensor, positions: torch.Tensor, inv_freq: torch.Tensor, dims: int) -> torch.Tensor:
    if dims == 0:
        return x
    a = positions.float()[:, None] * inv_freq[None]
    c, s = a.cos()[:, None], a.sin()[:, None]
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def qkv_prepare(proj: Branch, spec: WindowSpec, w: WindowWeights, positions: torch.Tensor, slots: torch.Tensor, cache: KVCache,
                layer: int) -> tuple[torch.Tensor, Optional[torch.Tensor]]:
    """Bias, norm over the whole query and key rows, rotation, store of keys and values at flat ``slots`` (negative = skip).
    Returns ``q [T, heads * maps * dq]`` and the sigmoid gates ``[T, heads]`` (fp32), if any."""
    src = proj.slabs if proj.slabs is not None else proj.rows
    T, dev = src.shape[-2], src.device
    nq, nk, nv = spec.q_cols, (0 if spec.shared else spec.k_cols), (0 if spec.shared else spec.v_cols)
    pages = cache.token_rows(layer)
    if not src.is_cuda:
        y = proj.value()
        if w.bias is not None:
            y = y + w.bias.float()
        q, k = y[:, :nq], y[:, nq:nq + nk]
        v = k if spec.tied else y[:, nq + nk:nq + nk + nv]

        def normed(z, weight, real):
            if spec.head_norm:
                h = z.reshape(T, -1, spec.dq)
                return (h / torch.sqrt(h.pow(2).sum(-1, keepdim=True) / spec.dim + spec.eps) * weight.float()).reshape(T, -1)
            return z / torch.sqrt(z.pow(2).sum(-1, keepdim=True) / real + spec.eps) * weight.float()

        if w.q_norm is not None:
            q = normed(q, w.q_norm, spec.heads * spec.maps * spec.dim)
            if nk:
                k = normed(k, w.k_norm, spec.kv_heads * spec.maps * spec.dim)
        q = _rotate(q.reshape(T, -1, spec.dq), positions, w.inv_freq, spec.rot_dims).reshape(T, nq)
        if nk:
            k = _rotate(k.reshape(T, -1, spec.dq), positions, w.inv_freq, spec.rot_dims).reshape(T, nk)
            keep = slots >= 0
            at = slots[keep]
            pages[at // cache.page, at % cache.page] = torch.cat([k, v], 1)[keep].to(pages.dtype)
        gate = torch.sigmoid(y[:, spec.gate_row:spec.gate_row + spec.heads]) if spec.gate else None
        return q.to(pages.dtype), gate
    assert positions.dtype == torch.int32 and positions.is_contiguous() and slots.dtype == torch.int64
    assert pages.shape[-1] == spec.k_cols + spec.v_cols and src.shape[-1] == spec.proj_cols
    q = torch.empty((T, nq), dtype=pages.dtype, device=dev)
    gate = torch.empty((T, spec.heads), dtype=torch.float32, device=dev) if spec.gate else None
    s, r = proj.slabs, proj.rows
    # a head's norm counts its own columns; without keys the key norm's weight is never read
    real = (spec.dim, spec.dim) if spec.head_norm else (spec.heads * spec.maps * spec.dim, spec.kv_heads * spec.maps * spec.dim)
    k_norm = w.k_norm if w.k_norm is not None or not spec.shared else w.q_norm
    native.call("prism_window_prepare", 1 if pages.dtype == torch.float32 else 0, _p(s), s.stride(0) if s is not None else 0,
                s.shape[0] if s is not None else 0, _p(r), r.stride(0) if r is not None else 0, _p(w.bias), _p(w.q_norm), _p(k_norm),
                _p(w.inv_freq), _p(positions), _p(slots), cache.num_blocks * cache.page, _p(q), _p(pages), _p(gate), T, spec.proj_cols,
                nq, nk, nv, spec.heads, spec.dq, spec.rot_dims, *real, 1 if spec.head_norm else 0, 1 if spec.tied else 0,
                float(spec.eps), _s(), _pdl())
    return q, gate


def _attention_cpu(q, spec, gate, sink, pages, page, block_tables, kv_lens, cu):
    T, H, G, M = q.shape[0], spec.heads, spec.kv_heads, spec.maps
    maps = torch.zeros((T, H, M, spec.dv))
    qh = q.float().view(T, G, H // G, M, spec.dq)
    for s, (lo, hi) in enumerate(zip(cu[:-1], cu[1:])):
        n = int(kv_lens[s])
        if n == 0:
            continue
        pos = torch.arange(n)
        blk = block_tables[s, pos // page].long()
        row = pages[blk.clamp_min(0), pos % page].float()
        k, v = row[:, :spec.k_cols].view(n, G, M, spec.dq), row[:, spec.k_cols:].view(n, G, spec.dv)
        at = torch.arange(n - (hi - lo), n)[:, None]
        seen = (pos <= at) & ((at - pos < spec.window) | (pos < spec.keep_first)) & (blk >= 0)
        sc = torch.einsum("tghmd,ngmd->tghmn", qh[lo:hi], k) * spec.scale
        if spec.softcap > 0.0:
            sc = spec.softcap * torch.tanh(sc / spec.softcap)
        sc = sc.masked_fill(~seen[:, None, None, None, :], float("-inf"))
        if sink is not None:
            sc = torch.cat([sc, sink.view(1, G, H // G, 1, 1).expand(hi - lo, -1, -1, -1, -1)], -1)
        p = torch.softmax(sc, -1)[..., :n]
        maps[lo:hi] = torch.einsum("tghmn,ngd->tghmd", p, v).reshape(hi - lo, H, M, spec.dv)
    o = maps[:, :, 0]
    if M == 2:
        o = o - spec.lam * maps[:, :, 1]
        o = o / torch.sqrt(o.pow(2).sum(-1, keepdim=True) / spec.vdim + spec.eps) * spec.gain
    if gate is not None:
        o = o * gate[:, :, None]
    return o.reshape(T, H * spec.dv).to(q.dtype)


def _decode_geometry(spec: WindowSpec, batch: int, reach: int) -> tuple[int, int]:
    """(16-row tiles per CTA, key splits): up to three CTAs per SM where the visible keys allow it."""
    rows = spec.heads // spec.kv_heads * spec.maps
    mt = 1 if rows <= 16 or spec.dv > 128 else 2
    blocks = batch * spec.kv_heads * -(-rows // (16 * mt))
    seen = min(reach, spec.window + KEY_TILE) + min(reach, spec.keep_first)
    tiles = max(1, -(-seen // KEY_TILE))
    return mt, max(1, min(MAX_SPLITS, tiles, 3 * SM_COUNT // max(1, blocks)))


def window_attention(q: torch.Tensor, spec: WindowSpec, gate: Optional[torch.Tensor], cache: KVCache, layer: int,
                     block_tables: torch.Tensor, kv_lens: torch.Tensor, *, cu_seqlens_q: Optional[torch.Tensor] = None,
                     max_q_len: int = 1, nsplit: int = 0, simple: bool = False, sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Attention of the new tokens ``q [T, heads * maps * dq]`` over the paged cache (their own rows already stored), combined
    over maps and gated: ``[T, heads * dv]``.  Without ``cu_seqlens_q`` every token is its own sequence (a decode step).
    ``simple``: the kernel that serves fp32 and any head width also for bf16."""
    T, H, M = q.shape[0], spec.heads, spec.maps
    pages = cache.token_rows(layer)
    if not q.is_cuda:
        cu = cu_seqlens_q.tolist() if cu_seqlens_q is not None else list(range(T + 1))
        return _attention_cpu(q, spec, gate, sink, pages, cache.page, block_tables, kv_lens, cu)
    assert block_tables.dtype == torch.int32 and kv_lens.dtype == torch.int32 and q.is_contiguous()
    assert sink is None or (sink.dtype == torch.float32 and sink.shape == (H,))
    S = T if cu_seqlens_q is None else cu_seqlens_q.shape[0] - 1
    out = torch.empty((T, H * spec.dv), dtype=q.dtype, device=q.device)
    head = (_p(q), _p(pages), _p(block_tables), _p(cu_seqlens_q), _p(kv_lens), _p(gate), _p(sink), _p(out), out.stride(0))
    sizes = (H, spec.kv_heads, M, spec.dq, spec.dv, spec.vdim, pages.shape[-1], cache.page, block_tables.shape[1], cache.num_blocks,
             spec.window, spec.keep_first)
    tail = (float(spec.scale), float(spec.lam), float(spec.gain), float(spec.eps), float(spec.softcap), _s(), _pdl())
    decode = cu_seqlens_q is None
    fast = not simple and q.dtype == torch.bfloat16
    if fast and decode and M * spec.dq <= MMA_MAX_KEY and spec.dv <= MMA_MAX_VALUE:
        mt, auto = _decode_geometry(spec, S, block_tables.shape[1] * cache.page)
        ns = nsplit if nsplit > 0 else auto
        rows = H // spec.kv_heads * M
        blocks = spec.kv_heads * -(-rows // (16 * mt))
        po = ml = counters = None
        if ns > 1:
            po = torch.empty((S * blocks * ns, 16 * mt, spec.dv), dtype=torch.float32, device=q.device)
            ml = torch.empty((S * blocks * ns, 16 * mt, 2), dtype=torch.float32, device=q.device)
            counters = _decode_counters(q.device, S * blocks)
        native.call("prism_window_decode", *head, _p(po), _p(ml), _p(counters), S, *sizes, mt, ns, *tail)
        return out
    if fast and not decode and spec.dq <= (TC_MAX_KEY if M == 1 else TC_MAX_HEAD) and spec.dv <= TC_MAX_HEAD and cache.page % 8 == 0 and spec.scale > 0.0:
        native.call("prism_window_prefill_tc", *head, T, S, int(max_q_len), *sizes, *tail)
        return out
    native.call("prism_window_attention_simple", 1 if q.dtype == torch.float32 else 0, *head, S, int(max_q_len), *sizes, *tail)
    return out


def token_side_gate(z: Branch, table: torch.Tensor, layer: int, ids: torch.Tensor) -> torch.Tensor:
    """``gelu_tanh(z) * table[ids, layer]``: ``z [T, D]``, ``table [vocab, layers, D]`` -> ``[T, D]`` of the table's type."""
    src = z.slabs if z.slabs is not None else z.rows
    T, D = src.shape[-2:]
    if not src.is_cuda:
        return (F.gelu(z.value(), approximate="tanh") * table[ids, layer].float()).to(table.dtype)
    assert table.is_contiguous() and ids.dtype == torch.int64 and D == table.shape[2] and D % 4 == 0
    out = torch.empty((T, D), dtype=table.dtype, device=table.device)
    s, r = z.slabs, z.rows
    native.call("prism_token_side_gate", 1 if table.dtype == torch.float32 else 0, _p(s), s.stride(0) if s is not None else 0,
                s.shape[0] if s is not None else 0, _p(r), r.stride(0) if r is not None else 0, _p(table), table.shape[0], table.stride(0),
                layer * D, _p(ids), _p(out), T, D, _s(), _pdl())
    return out
