"""Ops of models with latent attention, stacked projections and a 32-bit residual stream.

As with the package's other ops, CUDA tensors run the kernels of ``libprism_b200.so`` (bf16, or the
true 32-bit kernels when the tensors are fp32) and raise without them; CPU tensors run the plain-PyTorch
statement.  Kernels: ``csrc/residual_stream.cu``, ``csrc/latent_attention.cu``, ``csrc/gemm_f32.cu``, the
section epilogue of ``csrc/gemm_tcgen05.cu`` and the gated form of ``csrc/attention_tcgen05.cu``.
"""

from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional, Sequence

import torch
import torch.nn.functional as F

from . import SM_COUNT, KVCache, _p, _pdl, _s, choose_splits, linear, linear_partial, narrow_splits, native

ACTS = {None: 0, "gelu_tanh": 1, "gelu": 2, "sigmoid": 3, "softcap": 4, "decay": 5}
MAX_SPLITS = 64
MAX_LATENT = 1024       # widest latent row of the attention kernels
NO_WINDOW = 1 << 30
FLASH_MAX_HEAD = 128    # widest head of the tcgen05 prefill attention
EXPAND_MAX_SCRATCH_BYTES = 2 << 30
# up to here the absorb kernel sums and rotates the queries itself, once per 128 columns of the row; above, a kernel before it
ABSORB_ROTATES_TOKENS = 16


# ------------------------------------------------------------------------------ stacked projections
class Sections:
    """Row ranges of a stacked weight matrix: ``(rows, alpha, act)`` each; ``cap`` bounds ``softcap`` sections
    (``cap * tanh(v / cap)``); ``decay`` is ``exp(-exp(v))``."""

    def __init__(self, parts: Sequence[tuple[int, float, Optional[str]]], cap: float = 0.0) -> None:
        self.parts = [(int(r), float(a), act) for r, a, act in parts]
        self.cap = float(cap)
        n = len(self.parts)
        ends, total = [], 0
        for rows, _, _ in self.parts:
            total += rows
            ends.append(total)
        self.rows = total
        self.row_end = (ctypes.c_int * n)(*ends)
        self.alpha = (ctypes.c_float * n)(*(a for _, a, _ in self.parts))
        self.act = (ctypes.c_int * n)(*(ACTS[act] for _, _, act in self.parts))

    def args(self) -> tuple:
        return (len(self.parts), ctypes.addressof(self.row_end), ctypes.addressof(self.alpha), ctypes.addressof(self.act), self.cap)


def _apply(y: torch.Tensor, act: Optional[str], cap: float) -> torch.Tensor:
    if act == "gelu":
        return F.gelu(y)
    if act == "gelu_tanh":
        return F.gelu(y, approximate="tanh")
    if act == "sigmoid":
        return torch.sigmoid(y)
    if act == "decay":
        return torch.exp(-torch.exp(y))
    return cap * torch.tanh(y / cap) if act == "softcap" else y


def _two_per_sm(m: int, tokens: int) -> int:
    """Operand-ring depth of a decode-sized projection with more row tiles than SMs: two CTAs share an SM, so the last
    tiles do not wait for a whole second wave (29184 x 4096, one token: 59 -> 44 us; 128 tokens: 98 -> 67 us).
    0 = as deep as fits."""
    if tokens > 128 or -(-m // 128) <= SM_COUNT:
        return 0
    return 5 if tokens <= 32 else (4 if tokens <= 64 else 3)


def linear_sections(x: torch.Tensor, w: torch.Tensor, sections: Sections, *, bias: Optional[torch.Tensor] = None,
                    out_f32: bool = False, stages: int = 0) -> torch.Tensor:
    """``act_i(alpha_i * x @ w_i.T + bias_i)`` for every row section ``i`` of ``w``, side by side in one ``[T, M]``."""
    T, K = x.shape
    M = w.shape[0]
    assert sections.rows == M
    if not x.is_cuda:
        y = F.linear(x.float(), w.float())
        cols, parts = 0, []
        for rows, alpha, act in sections.parts:
            z = y[:, cols:cols + rows] * alpha
            if bias is not None:
                z = z + bias[cols:cols + rows].float()
            parts.append(_apply(z, act, sections.cap))
            cols += rows
        y = torch.cat(parts, dim=1)
        return y if out_f32 else y.to(x.dtype)
    assert x.stride(1) == 1 and w.stride(1) == 1 and x.dtype == w.dtype
    n, ends, alpha, act, cap = sections.args()
    if x.dtype == torch.float32:
        out = torch.empty((T, M), dtype=torch.float32, device=x.device)
        native.call("prism_gemm_f32", _p(w), _p(x), _p(out), M, T, K, w.stride(0), x.stride(0), out.stride(0), _p(bias), n, ends,
                    alpha, act, cap, _s(), _pdl())
        return out
    out = torch.empty((T, M), dtype=torch.float32 if out_f32 else torch.bfloat16, device=x.device)
    native.call("prism_gemm_wx_sections", _p(w), _p(x), _p(out), M, T, K, w.stride(0), x.stride(0), out.stride(0), _p(bias), n,
                ends, alpha, act, cap, 1 if out_f32 else 0, 0, stages or _two_per_sm(M, T), _s(), _pdl())
    return out


def linear_slabs(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """fp32 slabs ``[S, T, M]`` whose sum is ``x @ w.T``, for any number of tokens."""
    if x.is_cuda and x.dtype == torch.float32:
        T, K = x.shape
        out = torch.empty((1, T, w.shape[0]), dtype=torch.float32, device=x.device)
        native.call("prism_gemm_f32", _p(w), _p(x), _p(out), w.shape[0], T, K, w.stride(0), x.stride(0), out.stride(1), None, 0,
                    None, None, None, 0.0, _s(), _pdl())
        return out
    m, k, tokens = w.shape[0], w.shape[1], x.shape[0]
    return linear_partial(x, w, max(choose_splits(m, k, tokens), narrow_splits(m, k, tokens)) if x.is_cuda else 1)


# --------------------------------------------------------------------------------- residual stream
@dataclass
class Branch:
    """Output of a sublayer on its way into the stream: fp32 ``slabs [S, T, W]`` or ``rows [T, W]``, with an
    element-wise ``gate [T, W]``.  With ``pos [T, K]`` the slabs or rows are those of (token, slot) pairs instead and a
    token's value is the sum of ``weight[t, k]`` times row ``pos[t, k]`` (negative: nothing).  ``post_norm [W]``: the
    value is divided by its root mean square and multiplied by this weight before it is added.  ``self_weight [T]``: the
    stream's own row, as it was, joins the value with this weight."""

    slabs: Optional[torch.Tensor] = None
    rows: Optional[torch.Tensor] = None
    gate: Optional[torch.Tensor] = None
    pos: Optional[torch.Tensor] = None
    weight: Optional[torch.Tensor] = None
    post_norm: Optional[torch.Tensor] = None
    self_weight: Optional[torch.Tensor] = None

    def value(self) -> torch.Tensor:
        v = self.slabs.sum(0) if self.slabs is not None else self.rows.float()
        if self.pos is not None:
            v = (v[self.pos.long().clamp_min(0)] * torch.where(self.pos >= 0, self.weight, 0.0)[..., None]).sum(1)
        return v if self.gate is None else v * self.gate.float()


def stream_update(x: torch.Tensor, width: int, eps: float, *, keep: bool, ids: Optional[torch.Tensor] = None,
                  table: Optional[torch.Tensor] = None, a: Optional[Branch] = None, b: Optional[Branch] = None, mult: float = 1.0,
                  bias: Optional[torch.Tensor] = None, norm_weight: Optional[torch.Tensor] = None, norm_out: Optional[torch.Tensor] = None,
                  raw_out: Optional[torch.Tensor] = None, embed_out: Optional[torch.Tensor] = None, embed_mult: float = 1.0,
                  norm_offset: float = 0.0, history: Optional[torch.Tensor] = None, depth: int = 0,
                  depth_weight: Optional[torch.Tensor] = None, conv=None) -> None:
    """``x [T, W]`` (fp32, in place) ``= (x if keep) + embed_mult * table[ids] + mult * (a + b) + bias``, and what follows reads of
    it: ``norm_out`` the rows over their root mean square (``width`` real columns, the rest are zero), times
    ``norm_weight`` if given, ``raw_out`` the rows themselves, ``embed_out`` the embedding rows, each in its own type.
    Only ``a`` may consist of pairs or be normalised (``Branch.post_norm``).  ``norm_offset`` is added to the norm weights (1:
    weights stored around zero).  ``history [n, T, W]`` (fp32): the new ``x`` is kept as its row ``depth``, and with
    ``depth_weight [depth + 1]`` (fp32) becomes the weighted sum of rows ``0 .. depth`` before anything else reads it.  ``conv``
    (``recurrent.ConvStep``, one token per sequence): ``norm_out`` goes through it."""
    assert b is None or (b.pos is None and b.post_norm is None and b.self_weight is None)
    T, W = x.shape
    if not x.is_cuda:
        new = x.clone() if keep else torch.zeros_like(x)
        for branch in (a, b):
            if branch is not None:
                v = branch.value()
                if branch.self_weight is not None:
                    v = v + branch.self_weight[:, None] * x
                if branch.post_norm is not None:
                    v = v / torch.sqrt(v.pow(2).sum(-1, keepdim=True) / width + eps) * (norm_offset + branch.post_norm.float())
                new += mult * v
        if bias is not None:
            new += bias.float()
        if ids is not None:
            emb = table[ids].float() * embed_mult
            new += emb
            if embed_out is not None:
                embed_out.copy_(emb)
        if history is not None:
            history[depth].copy_(new)
            if depth_weight is not None:
                new = torch.einsum("j,jtw->tw", depth_weight, history[:depth + 1])
        x.copy_(new)
        if raw_out is not None:
            raw_out.copy_(new)
        if norm_out is not None:
            n = new / torch.sqrt(new.pow(2).sum(-1, keepdim=True) / width + eps)
            norm_out.copy_(n if norm_weight is None else n * (norm_offset + norm_weight.float()))
            if conv is not None:
                from .recurrent import short_conv

                norm_out.copy_(short_conv(norm_out, conv.weight, conv.spec, conv.state))
        return
    kinds = [t.dtype for t in (table, bias, norm_weight, norm_out, raw_out, embed_out) if t is not None]
    for branch in (a, b):
        if branch is not None:
            kinds += [t.dtype for t in (branch.rows, branch.gate, branch.post_norm) if t is not None]
    assert x.dtype == torch.float32 and x.is_contiguous() and len(set(kinds)) == 1
    gate_ld = 0
    flat: list = []
    for branch in (a, b):
        if branch is None:
            flat += [None, 0, 0, None, 0, None]
            continue
        s, r, g = branch.slabs, branch.rows, branch.gate
        assert s is None or (s.stride(1) == W and s.stride(2) == 1)
        if g is not None:
            assert gate_ld in (0, g.stride(0))
            gate_ld = g.stride(0)
        flat += [_p(s), s.stride(0) if s is not None else 0, s.shape[0] if s is not None else 0, _p(r),
                 r.stride(0) if r is not None else 0, _p(g)]
    ld = lambda t: t.stride(0) if t is not None else 0  # noqa: E731
    pairs = a is not None and a.pos is not None
    extra = (_p(a.pos) if pairs else None, _p(a.weight) if pairs else None, a.pos.shape[1] if pairs else 0,
             _p(a.post_norm) if a is not None else None, _p(a.self_weight) if a is not None else None)
    assert history is None or (history.dtype == torch.float32 and history.shape[1:] == x.shape and history[depth].is_contiguous())
    assert depth_weight is None or (depth_weight.dtype == torch.float32 and depth_weight.shape == (depth + 1,) and history is not None)
    assert conv is None or (conv.weight.dtype == norm_out.dtype and conv.weight.shape == (conv.spec.taps, W))
    behind = (_p(history), history.stride(0) if history is not None else 0, _p(depth_weight), depth,
              *(conv.args() if conv is not None else (None, 0, None, 0, 0, 0, None, None)))
    native.call("prism_stream_update", 1 if kinds[0] == torch.float32 else 0, T, _p(x), 1 if keep else 0, _p(ids), _p(table),
                table.shape[0] if table is not None else 0, *flat, gate_ld, *extra, float(mult), float(embed_mult), float(norm_offset), _p(bias), _p(norm_weight), _p(norm_out), ld(norm_out),
                _p(raw_out), ld(raw_out), _p(embed_out), ld(embed_out), W, width, float(eps), *behind, _s(),
                0 if ids is not None else _pdl())  # the first kernel of a step may follow a copy: full dependency


# -------------------------------------------------------------------------------- latent attention
@dataclass
class Rotary:
    """Rotation of neighbouring columns: pair ``i`` of a row at position ``p`` turns by ``p * inv_freq[i]``, sine and cosine times
    ``amplitude``.  ``start``: first of the ``dims`` columns in a query head, ``row_start`` in a cached row."""

    inv_freq: torch.Tensor   # [dims / 2] fp32
    dims: int
    start: int
    row_start: int
    amplitude: float = 1.0

    def apply(self, x: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
        """``x [T, ..., dims]`` turned, fp32 (the plain statement)."""
        a = (positions.float()[:, None] * self.inv_freq[None]).view(x.shape[0], *([1] * (x.dim() - 2)), -1)
        c, s = a.cos() * self.amplitude, a.sin() * self.amplitude
        u, v = x[..., 0::2].float(), x[..., 1::2].float()
        return torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2)

    def args(self, positions: torch.Tensor) -> tuple:
        assert positions.dtype == torch.int32 and positions.is_contiguous() and self.inv_freq.dtype == torch.float32
        return _p(self.inv_freq), _p(positions), float(self.amplitude)


NO_ROTARY = (None, None, 1.0)


@dataclass
class LatentWeights:
    """What a latent-attention layer multiplies latents with.  ``uk [H * dq, Rc]`` and ``uv [H * dv, Rc]`` are the two
    halves of ``ukv``; ``norm [R]`` is the latent's RMS-norm weight (padded to 16 where the layer's latents are made by
    ``latent_prepare``; none: another layer's are read).  ``dq`` / ``dv`` are the padded head widths, ``Rc`` the padded row
    width; padding is zero.  A rotated key part that all heads share lies behind the latent in the row (``rot``); ``uk`` has an
    identity block for it, so that a query's rotated columns meet it.  A query sees the ``window`` newest rows."""

    heads: int
    dq: int
    dv: int
    rank: int
    scale: float
    norm: Optional[torch.Tensor]
    ukv: torch.Tensor
    rot: Optional[Rotary] = None
    window: int = NO_WINDOW
    q_rank: int = 0
    q_norm: Optional[torch.Tensor] = None    # [q_rank padded to 16] of the query latent

    @property
    def uk(self) -> torch.Tensor:
        return self.ukv[:self.heads * self.dq]

    @property
    def uv(self) -> torch.Tensor:
        return self.ukv[self.heads * self.dq:]

    @property
    def value_cols(self) -> int:
        """Columns of a row that values are made of, in whole tiles."""
        return -(-self.rank // 64) * 64

    def connect_rotary(self) -> None:
        """The identity blocks of ``uk``."""
        if self.rot is not None:
            uk, i = self.uk.view(self.heads, self.dq, -1), torch.arange(self.rot.dims, device=self.ukv.device)
            uk[:, self.rot.start + i, self.rot.row_start + i] = 1.0


def latent_prepare(y: Branch, lw: LatentWeights, eps: float, positions: torch.Tensor, slots: torch.Tensor, cache: KVCache,
                   layer: int) -> torch.Tensor:
    """From the stacked projection ``y [T, query latent | key latent | shared key part]`` (sections padded to 16): the normalised
    query latent ``[T, Qp]``; normalised key latent and rotated key part go to the cache rows at flat ``slots`` (negative = skip).
    A layer that reads another's rows projects the query latent alone."""
    src = y.slabs if y.slabs is not None else y.rows
    T, Qp, Cp = src.shape[-2], lw.q_norm.shape[0], lw.norm.shape[0] if lw.norm is not None else 0
    pages = cache.latent(layer)
    if not src.is_cuda:
        v = y.value()

        def normed(z, real, weight):
            return z / torch.sqrt(z.pow(2).sum(-1, keepdim=True) / real + eps) * weight.float()

        if Cp:
            row = torch.zeros((T, pages.shape[-1]))
            row[:, :Cp] = normed(v[:, Qp:Qp + Cp], lw.rank, lw.norm)
            if lw.rot is not None:
                row[:, Cp:Cp + lw.rot.dims] = lw.rot.apply(v[:, Qp + Cp:Qp + Cp + lw.rot.dims], positions)
            at = slots[slots >= 0]
            pages[at // cache.page, at % cache.page] = row[slots >= 0].to(pages.dtype)
        return normed(v[:, :Qp], lw.q_rank, lw.q_norm).to(lw.q_norm.dtype)
    out = torch.empty((T, Qp), dtype=lw.q_norm.dtype, device=src.device)
    dims = lw.rot.dims if lw.rot is not None else 0
    assert slots.dtype == torch.int64 and src.shape[-1] >= Qp + Cp + (-(-dims // 4) * 4 if Cp else 0) and (lw.rot is None or lw.rot.row_start == Cp or not Cp)
    native.call("prism_latent_prepare", 1 if out.dtype == torch.float32 else 0, *_branch_args(y), _p(lw.q_norm), _p(lw.norm), _p(out), _p(pages),
                _p(slots), cache.num_blocks * cache.page, *(lw.rot.args(positions) if lw.rot is not None else NO_ROTARY), T, lw.q_rank, Qp, lw.rank,
                Cp, dims, pages.shape[-1], float(eps), _s(), _pdl())
    return out


def _branch_args(b: Branch) -> tuple:
    """(slabs, stride between them, their number, rows, stride between rows)"""
    s, r = b.slabs, b.rows
    assert s is None or s.stride(2) == 1
    return (_p(s), s.stride(0) if s is not None else 0, s.shape[0] if s is not None else 0, _p(r), s.stride(1) if s is not None else r.stride(0))


def rotate_queries(q: Branch, lw: LatentWeights, positions: torch.Tensor) -> torch.Tensor:
    """Queries ``[T, H * dq]`` of a projection with their rotated columns turned, in the weights' type; rows are turned in place."""
    src = q.slabs if q.slabs is not None else q.rows
    T, H, dtype = src.shape[-2], lw.heads, lw.ukv.dtype
    if not src.is_cuda:
        v = q.value().clone().view(T, H, lw.dq)
        if lw.rot is not None:
            part = v[..., lw.rot.start:lw.rot.start + lw.rot.dims]
            part.copy_(lw.rot.apply(part, positions))
        return v.view(T, H * lw.dq).to(dtype)
    out = torch.empty((T, H * lw.dq), dtype=dtype, device=src.device) if q.rows is None else q.rows
    start, dims = (lw.rot.start, lw.rot.dims) if lw.rot is not None else (0, 0)
    native.call("prism_latent_rotate", 1 if dtype == torch.float32 else 0, *_branch_args(q), _p(out), out.stride(0),
                *(lw.rot.args(positions) if lw.rot is not None else NO_ROTARY), T, H, lw.dq, start, dims, _s(), _pdl())
    return out


def latent_norm_store(raw: torch.Tensor, lw: LatentWeights, eps: float, slots: torch.Tensor, cache: KVCache, layer: int, *,
                      rows: Optional[torch.Tensor] = None) -> None:
    """RMS-normalise the projected latents ``raw [T, R]`` with their weight and store them at flat ``slots`` (negative =
    skip) of a single-plane cache, and into ``rows [T, Rc]`` when given."""
    T, Rc = raw.shape[0], cache.latent(layer).shape[-1]
    if not raw.is_cuda:
        v = raw[:, :lw.rank].float()
        c = v / torch.sqrt(v.pow(2).mean(-1, keepdim=True) + eps) * lw.norm.float()
        keep = slots >= 0
        pages = cache.latent(layer)
        pages[slots[keep] // cache.page, slots[keep] % cache.page, :lw.rank] = c[keep].to(pages.dtype)
        pages[slots[keep] // cache.page, slots[keep] % cache.page, lw.rank:] = 0
        if rows is not None:
            rows.zero_()
            rows[:, :lw.rank] = c.to(rows.dtype)
        return
    native.call("prism_latent_norm_store", 1 if raw.dtype == torch.float32 else 0, _p(raw), raw.stride(0), _p(lw.norm),
                _p(cache.latent(layer)), _p(slots), cache.num_blocks * cache.page, _p(rows), T, lw.rank, Rc, float(eps), _s(), _pdl())


def latent_splits(sequences: int, rows: int, reach: int = NO_WINDOW) -> int:
    """CTAs per key range: one CTA per SM is resident, so no more than fill the device once, nor than tiles in ``reach`` rows."""
    tiles = sequences * max(1, -(-rows // (16 if rows <= 16 else 32)))
    return max(1, min(MAX_SPLITS, SM_COUNT // tiles, -(-reach // 64) + 1))


def latent_attention_absorbed(
    q: "torch.Tensor | Branch", raw: Optional[torch.Tensor], gate: Optional[torch.Tensor], lw: LatentWeights, eps: float, slots: torch.Tensor,
    cache: KVCache, layer: int, block_tables: torch.Tensor, kv_lens: torch.Tensor, *, cu_seqlens_q: Optional[torch.Tensor] = None,
    max_q_len: int = 1, nsplit: int = 0, positions: Optional[torch.Tensor] = None,
) -> torch.Tensor:
    """Store the new tokens' latents (``raw``; none: they are in their pages already), then causal attention of their heads
    over the paged latents in the absorbed form, times the output ``gate``: ``[T, H * dv]``.

    ``q [T, H * dq]``, ``raw [T, R]`` and ``gate [T, H * dv]`` may be column ranges of a stacked projection; ``q`` may be a branch.
    Its rotated columns are turned here (``positions``).  Without ``cu_seqlens_q`` every token is its own sequence (a decode
    step)."""
    if isinstance(q, torch.Tensor):
        q = Branch(rows=q)
    src = q.slabs if q.slabs is not None else q.rows
    pages = cache.latent(layer)
    T, H, Rc, Rv = src.shape[-2], lw.heads, pages.shape[-1], lw.value_cols
    if raw is not None and (not src.is_cuda or lw.ukv.dtype == torch.float32):
        latent_norm_store(raw, lw, eps, slots, cache, layer)
    if not src.is_cuda:
        qa = torch.einsum("thd,hdr->thr", rotate_queries(q, lw, positions).view(T, H, lw.dq).float(), lw.uk.float().view(H, lw.dq, Rc))
        lat = torch.zeros((T, H, Rc), dtype=torch.float32)
        cu = cu_seqlens_q.tolist() if cu_seqlens_q is not None else list(range(T + 1))
        for s, (lo, hi) in enumerate(zip(cu[:-1], cu[1:])):
            n = int(kv_lens[s])
            if n == 0:
                continue
            pos = torch.arange(n)
            blk = block_tables[s, pos // cache.page].long()
            c = pages[blk.clamp_min(0), pos % cache.page].float()
            sc = torch.einsum("thr,nr->thn", qa[lo:hi], c) * lw.scale
            at = torch.arange(n - (hi - lo), n)[:, None]
            seen = (pos[None, :] <= at) & (at - pos[None, :] < lw.window) & (blk >= 0)[None, :]
            sc = sc.masked_fill(~seen[:, None, :], float("-inf"))
            lat[lo:hi] = torch.einsum("thn,nr->thr", torch.softmax(sc, dim=-1), c)
        o = torch.einsum("thr,hvr->thv", lat, lw.uv.float().view(H, lw.dv, Rc)).reshape(T, H * lw.dv)
        return (o if gate is None else o * gate.float()).to(lw.ukv.dtype)
    S = T if cu_seqlens_q is None else cu_seqlens_q.shape[0] - 1
    dev, dtype = src.device, lw.ukv.dtype
    page_args = (_p(pages), _p(block_tables), _p(cu_seqlens_q), _p(kv_lens))
    assert block_tables.dtype == torch.int32 and kv_lens.dtype == torch.int32 and slots.dtype == torch.int64
    gate_ld = gate.stride(0) if gate is not None else 0
    if dtype == torch.float32:
        rows = q.rows if lw.rot is None and q.rows is not None else rotate_queries(q, lw, positions)
        qa = torch.empty((T, H, Rc), dtype=torch.float32, device=dev)
        native.call("prism_headwise_f32", _p(rows), rows.stride(0), _p(lw.uk), Rc, None, 0, _p(qa), H * Rc, T, H, lw.dq, Rc, 0, _s(), _pdl())
        lat = torch.empty_like(qa)
        native.call("prism_latent_attention_f32", _p(qa), *page_args, _p(lat), S, max_q_len, H, Rc, cache.page, block_tables.shape[1],
                    cache.num_blocks, lw.window, float(lw.scale), _s(), _pdl())
        out = torch.empty((T, H * lw.dv), dtype=torch.float32, device=dev)
        native.call("prism_headwise_f32", _p(lat), H * Rc, _p(lw.uv), Rc, _p(gate), gate_ld, _p(out), H * lw.dv, T, H, Rc, lw.dv, 1,
                    _s(), _pdl())
        return out
    if nsplit <= 0:
        nsplit = latent_splits(S, max_q_len * H, lw.window + max_q_len)
    turned = lw.rot is None
    if T > ABSORB_ROTATES_TOKENS and (lw.rot is not None or q.rows is None):
        q, turned = Branch(rows=rotate_queries(q, lw, positions)), True
    qa = torch.empty((T, H, Rc), dtype=torch.bfloat16, device=dev)
    rot = (*NO_ROTARY, 0, 0) if turned else (*lw.rot.args(positions), lw.rot.start, lw.rot.dims)
    slabs, stride, P, rows, ld = _branch_args(q)
    native.call("prism_latent_absorb", rows, slabs, stride, P, ld, *rot, _p(lw.uk), _p(qa), _p(raw), raw.stride(0) if raw is not None else 0,
                _p(lw.norm), _p(pages), _p(slots), cache.num_blocks * cache.page, T, H, lw.dq, lw.rank, Rc, float(eps), _s(), _pdl())
    part_o = part_ml = lat = None
    if nsplit > 1:
        part_o = torch.empty((T * H, nsplit, Rv), dtype=torch.float32, device=dev)
        part_ml = torch.empty((T * H, nsplit, 2), dtype=torch.float32, device=dev)
    else:
        lat = torch.empty((T * H, Rv), dtype=torch.bfloat16, device=dev)
    native.call("prism_latent_attention", _p(qa), *page_args, _p(part_o), _p(part_ml), _p(lat), S, max_q_len, H, Rc, Rv, cache.page,
                block_tables.shape[1], cache.num_blocks, nsplit, lw.window, float(lw.scale), _s(), _pdl())
    out = torch.empty((T, H * lw.dv), dtype=torch.bfloat16, device=dev)
    native.call("prism_latent_out", _p(part_o), _p(part_ml), _p(lat), _p(lw.uv), Rc, _p(gate), gate_ld, _p(out), out.stride(0), T, H, lw.dv,
                Rv, nsplit, _s(), _pdl())
    return out


def expanded_is_cheaper(lw: LatentWeights, row: int, total_kv: int, attended_pairs: int) -> bool:
    """Whether a prompt step runs faster with explicit keys and values.  Per attended pair the absorbed form
    multiplies 2 x ``row`` elements per head, the expanded form ``dq + dv``, on a tensor-core path that is about
    2.5 times as fast, but it first makes keys and values of every visible latent."""
    if lw.dq != lw.dv or lw.dq > FLASH_MAX_HEAD:
        return False
    if total_kv * 2 * (row + lw.heads * (lw.dq + lw.dv)) > EXPAND_MAX_SCRATCH_BYTES:
        return False
    absorbed = attended_pairs * 2 * row
    expanded = (attended_pairs + total_kv * row) * (lw.dq + lw.dv)
    return expanded < 2.5 * absorbed


def latent_attention_expanded(
    q: torch.Tensor, raw: torch.Tensor, gate: Optional[torch.Tensor], lw: LatentWeights, eps: float, slots: torch.Tensor,
    cache: KVCache, layer: int, block_tables: torch.Tensor, cu_seqlens_q: torch.Tensor, max_q_len: int, *,
    cu_seqlens_kv: Optional[torch.Tensor] = None, total_kv: int = 0, max_kv_len: int = 0,
) -> torch.Tensor:
    """The same result from explicit keys and values (bf16, CUDA): the visible latents as contiguous rows (the new
    tokens' own without ``cu_seqlens_kv``, else gathered from their pages), one GEMM for the keys and values of all
    heads, and the tcgen05 attention kernel with the gate in its epilogue."""
    T, H, Rc = q.shape[0], lw.heads, cache.latent(layer).shape[-1]
    dev, S = q.device, cu_seqlens_q.shape[0] - 1
    assert q.is_cuda and q.dtype == torch.bfloat16 and lw.dq == lw.dv
    total = T if cu_seqlens_kv is None else int(total_kv)
    c = torch.empty((total, Rc), dtype=torch.bfloat16, device=dev)
    latent_norm_store(raw, lw, eps, slots, cache, layer, rows=c if cu_seqlens_kv is None else None)
    if cu_seqlens_kv is not None:
        native.call("prism_gather_latents", _p(cache.latent(layer)), _p(block_tables), _p(cu_seqlens_kv), _p(c), S, int(max_kv_len),
                    total, block_tables.shape[1], cache.num_blocks, cache.page, Rc * 2, _s(), _pdl())
    kv = linear(c, lw.ukv)
    k, v = kv[:, :H * lw.dq], kv[:, H * lw.dq:]
    out = torch.empty((T, H * lw.dv), dtype=torch.bfloat16, device=dev)
    native.call("prism_flash_attention_tc_kv", _p(q), q.stride(0), _p(k), _p(v), kv.stride(0), _p(out), out.stride(0),
                _p(cu_seqlens_q), _p(cu_seqlens_kv), _p(gate), gate.stride(0) if gate is not None else 0, T, total, S, int(max_q_len),
                H, H, lw.dq, float(lw.scale), _s(), _pdl())
    return out


# ------------------------------------------------------------------------- explicit keys of a window
@dataclass
class ExpandPlan:
    """Where a prompt step's explicit keys and values go: of every sequence the pages that its new tokens see, from ``first[s]``
    on, become scratch pages ``base[s] ..``; ``table`` is the block table of the scratch."""

    first: torch.Tensor      # [S] int32
    base: torch.Tensor       # [S + 1] int32
    table: torch.Tensor      # [S, max_blocks] int32
    pages: int
    max_pages: int
    pairs: int               # (new token, visible row) pairs, rounded up to tiles

    @classmethod
    def make(cls, lens: Sequence[tuple[int, int]], window: int, page: int, max_blocks: int, device) -> "ExpandPlan":
        """``lens``: (new tokens, tokens up to the last of them) per sequence."""
        S = len(lens)
        host = torch.full((S, max_blocks), -1, dtype=torch.int32)
        marks = torch.zeros((2, S + 1), dtype=torch.int32)
        most = pairs = 0
        for s, (n, kv) in enumerate(lens):
            first, stop = (max(0, kv - n - window + 1) // page, -(-kv // page)) if n > 0 else (0, 0)
            base = int(marks[1, s])
            marks[0, s], marks[1, s + 1] = first, base + stop - first
            host[s, first:stop] = torch.arange(base, base + stop - first, dtype=torch.int32)
            most, pairs = max(most, stop - first), pairs + n * min(kv, window + 63)

        def put(t: torch.Tensor) -> torch.Tensor:
            return t if torch.device(device).type == "cpu" else t.pin_memory().to(device, non_blocking=True)

        marks_d = put(marks)
        return cls(marks_d[0, :S], marks_d[1], put(host), int(marks[1, S]), most, pairs)

    def is_cheaper(self, lw: LatentWeights, row: int, page: int) -> bool:
        """Whether explicit keys and values beat the absorbed form.  Per pair that multiplies ``row`` and the latent's elements
        per head, the explicit form ``dq + dv`` on a tensor-core path that is about 2.5 times as fast, behind a projection of
        every visible row."""
        from .window import TC_MAX_HEAD, TC_MAX_KEY

        rows, width = self.pages * page, lw.dq + lw.dv
        if lw.dq > TC_MAX_KEY or lw.dq % 16 or lw.dv > TC_MAX_HEAD or lw.dv % 16 or page % 8 or lw.scale <= 0.0:
            return False
        if rows * 2 * (row + lw.heads * width) > EXPAND_MAX_SCRATCH_BYTES:
            return False
        return (self.pairs + rows * row) * width < 2.5 * self.pairs * (row + lw.value_cols)


@dataclass
class _ScratchPages:
    """Scratch rows as the attention over single-row caches sees a cache."""

    rows: torch.Tensor       # [blocks, page, row]

    def token_rows(self, layer: int) -> torch.Tensor:
        return self.rows

    @property
    def num_blocks(self) -> int:
        return self.rows.shape[0]

    @property
    def page(self) -> int:
        return self.rows.shape[1]


def latent_attention_windowed(q: torch.Tensor, lw: LatentWeights, cache: KVCache, layer: int, block_tables: torch.Tensor, kv_lens: torch.Tensor,
                              cu_seqlens_q: torch.Tensor, max_q_len: int, plan: ExpandPlan) -> torch.Tensor:
    """Attention of rotated queries ``q [T, H * dq]`` (bf16, CUDA) with explicit keys and values: the visible rows gathered page by
    page, one GEMM for the keys and values of all heads, and the tcgen05 attention over paged rows with a window."""
    from .window import WindowSpec, window_attention

    pages = cache.latent(layer)
    H, Rc, page, rows = lw.heads, pages.shape[-1], cache.page, plan.pages * cache.page
    c = torch.empty((rows, Rc), dtype=torch.bfloat16, device=q.device)
    native.call("prism_gather_latent_pages", _p(pages), _p(block_tables), _p(kv_lens), _p(plan.first), _p(plan.base), _p(c), kv_lens.shape[0],
                plan.max_pages, rows, block_tables.shape[1], cache.num_blocks, page, Rc * 2, _s(), _pdl())
    kv = _ScratchPages(linear(c, lw.ukv).view(plan.pages, page, H * (lw.dq + lw.dv)))
    spec = WindowSpec(heads=H, kv_heads=H, maps=1, dim=lw.dq, vdim=lw.dv, rot_dims=0, scale=lw.scale, window=lw.window, keep_first=0, gate=False,
                      eps=0.0)
    return window_attention(q, spec, None, kv, 0, plan.table, kv_lens, cu_seqlens_q=cu_seqlens_q, max_q_len=max_q_len)
