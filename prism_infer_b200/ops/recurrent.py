"""Recurrent state of sequences, recurrences with a matrix state per head, and the short convolution in front of a mixer.

A sequence's state lives in a slot: per recurrent layer a row of fp32, in two versions.  A step that takes a sequence from
``c`` tokens to ``c'`` reads version ``c & 1`` and writes version ``c' & 1``; a step that is run again (a decode launch that ran
ahead and was not taken over) finds what it read before.  A sequence without tokens starts from zero, whatever the slot holds.

With ``h'`` the previous token's row, every projection reads its own blend ``h + (h' - h) * mu``; per head, with receptance
``r``, key ``k``, value ``v``, decay ``d = exp(-exp(w0 + W2 tanh(W1 blend)))`` and bonus ``u``:

    o_t = (S + diag(u) k v^T)^T r        S <- diag(d) S + k v^T

and the mixer's output is ``o`` over its root mean square per head, times a weight, times ``silu`` of the gate.

The forget rule has no keys: a gate per head and key channel, ``f = l + (1 - l) sigmoid(z + b)`` above a learned bound ``l``, decays
the state and weighs what is written; the query ``q = silu(y)`` reads behind the update:

    S <- diag(f) S + (1 - f) v^T        o_t = S^T q

and the output is ``o`` over its root mean square per head, times a weight that all heads share.

The short convolution adds a causal sum over the last ``taps`` rows of every channel to a row; the last ``taps - 1`` rows are
carried on in the state.

CUDA tensors run the kernels of ``csrc/recurrence.cu`` and raise without them; CPU tensors run the plain-PyTorch statement.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Sequence

import torch
import torch.nn.functional as F

from . import SM_COUNT, _p, _pdl, _s, effective_splits, native
from .latent import Branch, Sections, linear_sections, linear_slabs

SMALL_TOKENS = 128      # up to here the four wide projections are one grouped split-K launch
TILE_ROWS, TILE_ROWS_F32 = 128, 64
MAX_HEAD = 256


class StateCache:
    """State slots of every recurrent layer: ``layer(i)`` is ``[slots, 2 versions, sizes[i]]`` fp32."""

    def __init__(self, sizes: Sequence[int], slots: int, device, pin_memory: bool = False) -> None:
        self.sizes, self.slots = tuple(int(s) for s in sizes), int(slots)
        kw = dict(device="cpu", pin_memory=True) if pin_memory else dict(device=device)
        self._layers = [torch.zeros((self.slots, 2, n), dtype=torch.float32, **kw) for n in self.sizes]

    def layer(self, i: int) -> torch.Tensor:
        return self._layers[i]

    def copy_slot(self, src: "StateCache", src_slot: int, dst_slot: int) -> None:
        """All layers and both versions of one slot, in stream order."""
        for d, s in zip(self._layers, src._layers):
            d[dst_slot].copy_(s[src_slot], non_blocking=True)

    def bytes(self) -> int:
        return sum(t.numel() * 4 for t in self._layers)


@dataclass(frozen=True)
class TimeMixSpec:
    """Sizes of one mixer.  ``n`` is ``dim`` padded to a multiple of 16 with zeros, ``rank`` the padded rank of the decay."""

    heads: int
    dim: int
    rank: int
    width: int               # padded width of the input rows
    eps: float

    @property
    def n(self) -> int:
        return -(-self.dim // 16) * 16

    @property
    def cols(self) -> int:
        return self.heads * self.n

    @property
    def carry(self) -> int:
        """Where the last token's row starts in a state row."""
        return self.heads * self.n * self.n


@dataclass
class TimeMixWeights:
    mu: torch.Tensor         # [5, W] blends of r, k, v, gate, decay
    rkvg: torch.Tensor       # [4, H n, W]
    w1: torch.Tensor         # [rank, W]
    w2: torch.Tensor         # [H n, rank]
    w0: torch.Tensor         # [H n]
    u: torch.Tensor          # [H n]
    norm: torch.Tensor       # [H n]

    def __post_init__(self) -> None:
        self._decay = Sections([(self.w2.shape[0], 1.0, "decay")])


@dataclass
class StateView:
    """The slots of a step's sequences in one layer."""

    cache: StateCache
    layer: int
    slots: torch.Tensor                            # [S] int32, negative: no state
    kv_lens: torch.Tensor                          # [S] int32 tokens up to and including the step's last
    cu_seqlens_q: Optional[torch.Tensor] = None    # [S + 1] int32; None: one token per sequence

    def args(self, spec: "TimeMixSpec | ForgetSpec | ConvSpec", cu: bool = True) -> tuple:
        t = self.cache.layer(self.layer)
        assert t.shape[2] >= spec.carry + spec.width and self.slots.dtype == torch.int32 and self.kv_lens.dtype == torch.int32
        return (_p(t), t.shape[2], t.shape[0], spec.carry, _p(self.slots)) + ((_p(self.cu_seqlens_q),) if cu else ()) + (_p(self.kv_lens),)


def _spans(st: StateView, tokens: int):
    """(sequence, slot, first token, end token, tokens before) of the sequences that have a slot."""
    cu = st.cu_seqlens_q.tolist() if st.cu_seqlens_q is not None else list(range(tokens + 1))
    for i, (lo, hi) in enumerate(zip(cu[:-1], cu[1:])):
        slot, end = int(st.slots[i]), int(st.kv_lens[i])
        if slot >= 0 and hi > lo:
            yield slot, lo, hi, end - (hi - lo)


def _time_mix_cpu(x: torch.Tensor, spec: TimeMixSpec, w: TimeMixWeights, st: StateView) -> torch.Tensor:
    dtype, H, n = w.rkvg.dtype, spec.heads, spec.n
    rows = st.cache.layer(st.layer)
    out = torch.zeros((x.shape[0], spec.cols), dtype=dtype)
    for slot, lo, hi, before in _spans(st, x.shape[0]):
        old = rows[slot, before & 1].clone() if before > 0 else torch.zeros(rows.shape[2])
        h = x[lo:hi]
        prev = torch.cat([old[None, spec.carry:], h[:-1]])
        mixed = [(h + (prev - h) * w.mu[m].float()).to(dtype) for m in range(5)]
        r, k, v, g = (F.linear(mixed[m].float(), w.rkvg[m].float()).view(-1, H, n) for m in range(4))
        t = torch.tanh(F.linear(mixed[4].float(), w.w1.float()))
        d = torch.exp(-torch.exp(F.linear(t, w.w2.float()) + w.w0.float())).view(-1, H, n)
        u = w.u.float().view(H, n)
        S = old[:spec.carry].view(H, n, n)
        o = torch.empty_like(r)
        for i in range(hi - lo):
            kv = k[i, :, :, None] * v[i, :, None, :]
            o[i] = ((S + u[:, :, None] * kv) * r[i, :, :, None]).sum(1)
            S = d[i, :, :, None] * S + kv
        o = o / torch.sqrt(o.pow(2).sum(-1, keepdim=True) / spec.dim + spec.eps)
        out[lo:hi] = (o.reshape(-1, spec.cols) * w.norm.float() * F.silu(g).reshape(-1, spec.cols)).to(dtype)
        new = rows[slot, (before + hi - lo) & 1]
        new[:spec.carry] = S.reshape(-1)
        new[spec.carry:] = h[-1]
    return out


def _proj_args(p: Branch) -> tuple:
    s, r = p.slabs, p.rows
    return (_p(s), s.stride(0) if s is not None else 0, s.shape[0] if s is not None else 0, _p(r),
            s.stride(1) if s is not None else r.stride(0))


def token_mix(x: torch.Tensor, spec: TimeMixSpec, w: TimeMixWeights, st: StateView):
    """``[5, T, W]`` blends of every row with the one before it, and the (table, entries, count) of their grouped projection."""
    T = x.shape[0]
    f32 = w.mu.dtype == torch.float32
    tile = TILE_ROWS_F32 if f32 else TILE_ROWS
    assert x.is_contiguous() and x.dtype == torch.float32 and x.shape[1] == spec.width
    mixed = torch.empty((5, T, spec.width), dtype=w.mu.dtype, device=x.device)
    entries = 4 * -(-T // tile)
    table = torch.empty((entries + 1, 4), dtype=torch.int32, device=x.device)   # its last row holds the count
    native.call("prism_token_mix", 1 if f32 else 0, *st.args(spec), _p(x), st.slots.shape[0], spec.width, _p(w.mu), _p(mixed), T, _p(table),
                _p(table[entries]), tile, _s(), _pdl())
    return mixed, (_p(table), entries, _p(table[entries])), table


def _grouped_splits(m: int, k: int) -> int:
    kb = -(-k // 64)
    return max(1, min(SM_COUNT // (4 * -(-m // 128)), kb // 4 if kb >= 8 else 1, 8))


def wide_projections(mixed: torch.Tensor, w: torch.Tensor, table: tuple) -> Branch:
    """The first four blends times their own matrices ``w [4, M, W]``, all rows one after another ``[4 T, M]``: one launch."""
    _, T, W = mixed.shape
    M, N = w.shape[1], 4 * T
    if w.dtype == torch.float32:
        y = torch.empty((1, N, M), dtype=torch.float32, device=w.device)
        native.call("prism_gemm_f32_grouped", _p(w), _p(mixed), _p(y), M, N, W, W, W, M, *table, None, N, 4, _s(), _pdl())
        return Branch(slabs=y)
    if T <= SMALL_TOKENS:
        splits = effective_splits(W, _grouped_splits(M, W))
        y = torch.empty((splits, N, M), dtype=torch.float32, device=w.device)
        native.call("prism_gemm_grouped_small", _p(w), _p(mixed), _p(y), M, T, N, W, W, M, *table, None, N, 4, 0, 0.0, splits, y.stride(0), _s(),
                    _pdl())
        return Branch(slabs=y)
    y = torch.empty((N, M), dtype=torch.bfloat16, device=w.device)
    native.call("prism_gemm_grouped", _p(w), _p(mixed), _p(y), M, N, W, W, M, *table, 4, 0, 0.0, _s(), _pdl())
    return Branch(rows=y)


def decays(z: torch.Tensor, w: TimeMixWeights) -> torch.Tensor:
    """``exp(-exp(w0 + W2 tanh(z)))`` in 32-bit, ``[T, H n]``, of the narrow projection's slabs ``z [S, T, rank]``."""
    _, T, R = z.shape
    C = w.w2.shape[0]
    if w.w2.dtype == torch.float32:
        t = torch.empty((T, R), dtype=torch.float32, device=z.device)
        native.call("prism_tanh_f32", _p(z), z.stride(0), z.shape[0], _p(t), T, R, _s(), _pdl())
        return linear_sections(t, w.w2, w._decay, bias=w.w0, out_f32=True)
    d = torch.empty((T, C), dtype=torch.float32, device=z.device)
    native.call("prism_decay_project", _p(z), z.stride(0), z.shape[0], z.stride(1), _p(w.w2), _p(w.w0), _p(d), T, C, R, _s(), _pdl())
    return d


def time_mix(x: torch.Tensor, spec: TimeMixSpec, w: TimeMixWeights, st: StateView) -> torch.Tensor:
    """The mixer up to its output projection for the step's rows ``x [T, W]`` (fp32): ``[T, H n]``, with the state taken from and
    put back into the sequences' slots.  Rows of sequences without a slot are zero."""
    if not x.is_cuda:
        return _time_mix_cpu(x, spec, w, st)
    T, S = x.shape[0], st.slots.shape[0]
    dtype, dev = w.rkvg.dtype, x.device
    f32 = 1 if dtype == torch.float32 else 0
    if spec.n > MAX_HEAD:
        raise ValueError(f"time mixing: heads of up to {MAX_HEAD} channels, got {spec.dim}")
    mixed, table, _keep = token_mix(x, spec, w, st)
    p = wide_projections(mixed, w.rkvg, table)
    z1 = linear_slabs(mixed[4], w.w1)
    out = torch.empty((T, spec.cols), dtype=dtype, device=dev)
    if st.cu_seqlens_q is None:
        native.call("prism_state_step", f32, *st.args(spec, cu=False), _p(x), S, spec.width, *_proj_args(p), *_proj_args(Branch(slabs=z1)),
                    _p(w.w2), _p(w.w0), _p(w.u), _p(w.norm), _p(out), spec.heads, spec.n, spec.dim, spec.rank, float(spec.eps), _s(), _pdl())
        return out
    d = decays(z1, w)
    o = torch.empty((T, spec.cols), dtype=torch.float32, device=dev)
    native.call("prism_state_scan", f32, *st.args(spec), _p(x), S, spec.width, *_proj_args(p), _p(d), _p(w.u), _p(o), T, spec.heads, spec.n,
                _s(), _pdl())
    native.call("prism_head_norm_gate", f32, _p(o), *_proj_args(p), _p(w.norm), _p(out), T, spec.heads, spec.n, spec.dim, float(spec.eps), _s(),
                _pdl())
    return out


# ----------------------------------------------------------------------------------------- the forget rule
@dataclass(frozen=True)
class ForgetSpec:
    """Sizes of one mixer: ``dim`` key and ``vdim`` value channels per head, padded to multiples of 16 (``n``, ``m``)."""

    heads: int
    dim: int
    vdim: int
    eps: float

    width = 0                # it carries no input row on

    @property
    def n(self) -> int:
        return -(-self.dim // 16) * 16

    @property
    def m(self) -> int:
        return -(-self.vdim // 16) * 16

    @property
    def gate_col(self) -> int:
        """First gate column of the stacked projection ``[queries | gates | values]``; ``value_col`` the first value column."""
        return self.heads * self.n

    @property
    def value_col(self) -> int:
        return 2 * self.heads * self.n

    @property
    def proj_cols(self) -> int:
        return self.heads * (2 * self.n + self.m)

    @property
    def carry(self) -> int:
        """Elements of the state; what a layer carries on besides starts there."""
        return self.heads * self.n * self.m


@dataclass
class ForgetWeights:
    bias: torch.Tensor       # [H n] of the gates
    lower: torch.Tensor      # [H n] bounds of the gates; one in padded channels, which then hold nothing
    norm: torch.Tensor       # [m]


def _forget_cpu(y: torch.Tensor, spec: ForgetSpec, w: ForgetWeights, st: StateView) -> torch.Tensor:
    H, n, m = spec.heads, spec.n, spec.m
    rows = st.cache.layer(st.layer)
    out = torch.zeros((y.shape[0], H * m), dtype=w.norm.dtype)
    for slot, lo, hi, before in _spans(st, y.shape[0]):
        q = F.silu(y[lo:hi, :spec.gate_col]).view(-1, H, n)
        keep = (1.0 - w.lower.float()) * torch.sigmoid(-(y[lo:hi, spec.gate_col:spec.value_col] + w.bias.float()))
        keep = keep.view(-1, H, n)
        v = y[lo:hi, spec.value_col:].view(-1, H, m)
        S = rows[slot, before & 1, :spec.carry].clone().view(H, n, m) if before > 0 else torch.zeros(H, n, m)
        o = torch.empty((hi - lo, H, m))
        for i in range(hi - lo):
            S = (1.0 - keep[i])[:, :, None] * S + keep[i, :, :, None] * v[i, :, None, :]
            o[i] = (S * q[i, :, :, None]).sum(1)
        o = o / torch.sqrt(o.pow(2).sum(-1, keepdim=True) / spec.vdim + spec.eps) * w.norm.float()
        out[lo:hi] = o.reshape(-1, H * m).to(out.dtype)
        rows[slot, (before + hi - lo) & 1, :spec.carry] = S.reshape(-1)
    return out


def forget_mix(p: Branch, spec: ForgetSpec, w: ForgetWeights, st: StateView) -> torch.Tensor:
    """The mixer up to its output projection for the step's stacked projection ``p [T, proj_cols]``: ``[T, H m]``, with the state
    taken from and put back into the sequences' slots.  Rows of sequences without a slot are zero."""
    src = p.slabs if p.slabs is not None else p.rows
    if not src.is_cuda:
        return _forget_cpu(p.value(), spec, w, st)
    if max(spec.n, spec.m) > MAX_HEAD:
        raise ValueError(f"gated linear attention: heads of up to {MAX_HEAD} channels, got {spec.dim} x {spec.vdim}")
    T, S, dev = src.shape[-2], st.slots.shape[0], src.device
    assert src.shape[-1] == spec.proj_cols and src.stride(-1) == 1
    f32 = 1 if w.norm.dtype == torch.float32 else 0
    out = torch.empty((T, spec.heads * spec.m), dtype=w.norm.dtype, device=dev)
    if st.cu_seqlens_q is None:
        native.call("prism_forget_step", f32, *st.args(spec, cu=False), S, *_proj_args(p), _p(w.bias), _p(w.lower), _p(w.norm), _p(out), spec.heads,
                    spec.n, spec.m, spec.vdim, float(spec.eps), _s(), _pdl())
        return out
    o = torch.empty((T, spec.heads * spec.m), dtype=torch.float32, device=dev)
    native.call("prism_forget_scan", f32, *st.args(spec), S, *_proj_args(p), _p(w.bias), _p(w.lower), _p(o), T, spec.heads, spec.n, spec.m, _s(),
                _pdl())
    native.call("prism_head_norm_gate", f32, _p(o), None, 0, 0, None, 0, _p(w.norm), _p(out), T, spec.heads, spec.m, spec.vdim, float(spec.eps),
                _s(), _pdl())
    return out


# ---------------------------------------------------------------------------------- the short convolution
MAX_TAPS = 16


@dataclass(frozen=True)
class ConvSpec:
    """``taps`` rows of ``row`` columns; those carried on start at element ``carry`` of the state row."""

    taps: int
    row: int
    carry: int

    @property
    def width(self) -> int:
        return (self.taps - 1) * self.row


@dataclass
class ConvStep:
    """The convolution of one token per sequence as a part of the kernel that makes its input rows (``stream_update``)."""

    weight: torch.Tensor     # [taps, W]
    spec: ConvSpec
    state: StateView

    def args(self) -> tuple:
        t = self.state.cache.layer(self.state.layer)
        _, row, slots, carry, slot_p, lens_p = self.state.args(self.spec, cu=False)
        return (_p(self.weight), self.spec.taps, _p(t), row, slots, carry, slot_p, lens_p)


def short_conv(x: torch.Tensor, weight: torch.Tensor, spec: ConvSpec, st: StateView, *, max_len: int = 1) -> torch.Tensor:
    """``x_t + sum_j weight[j] x_(t - taps + 1 + j)`` for the step's rows ``x [T, W]``, the rows before them from the sequences'
    slots, whose carry is renewed.  ``max_len``: the most tokens of a sequence."""
    if spec.taps > MAX_TAPS:
        raise ValueError(f"convolutions of up to {MAX_TAPS} taps, got {spec.taps}")
    keep = spec.taps - 1
    if not x.is_cuda:
        rows, out = st.cache.layer(st.layer), x.clone()
        for slot, lo, hi, before in _spans(st, x.shape[0]):
            old = rows[slot, before & 1, spec.carry:spec.carry + spec.width].clone().view(keep, spec.row)
            seen = torch.cat([old if before > 0 else torch.zeros_like(old), x[lo:hi].float()])
            n = hi - lo
            out[lo:hi] = (x[lo:hi].float() + sum(weight[j].float() * seen[j:j + n] for j in range(spec.taps))).to(x.dtype)
            rows[slot, (before + n) & 1, spec.carry:spec.carry + spec.width] = seen[n:].reshape(-1)
        return out
    assert x.is_contiguous() and weight.is_contiguous() and x.dtype == weight.dtype and x.shape[1] == spec.row and st.cu_seqlens_q is not None
    out = torch.empty_like(x)
    native.call("prism_short_conv", 1 if x.dtype == torch.float32 else 0, *st.args(spec), st.slots.shape[0], spec.row, _p(x), _p(weight), _p(out),
                spec.taps, int(max_len), _s(), _pdl())
    return out
