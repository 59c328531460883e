"""Fosulix: a decoder that alternates gated linear attention with windowed latent attention, all feed-forwards routed, every
mixer behind a short convolution and every layer behind an average over the depth, as the engine runs it.

With ``N_w(y)`` a row over its root mean square times ``w`` and ``X_0`` the embedding rows, layer ``i`` is

    h = N_1(x)                      h += short convolution of h over the last few tokens, channel by channel
    x += m mixer(h)
    x += m experts(N_2(x))          if the layer has a feed-forward
    X_(i+1) = x                     x = sum_j a_ij X_j,  j = 0 .. i + 1

The mixers:

    hgrn2               a matrix state per head; one gate per key channel decays and writes (``ops/recurrent.py``)
    latent_attention    queries and keys through normalised latents, a rotated key part that all heads share, a window; a layer may
                        read the cached rows of an earlier one instead of its own (``ops/latent.py``)

The residual ``x`` and the kept results ``X_j`` stay fp32.  One kernel adds a branch, keeps the result, averages, normalises and,
in a decode step, runs the convolution in front of the next mixer.  Every layer has a row of state: its recurrent state, if any,
then the rows its convolution carries on.  Cache slabs exist for the layers with latents of their own.  Decode steps and short
portions attend in the absorbed form over the cached rows; longer ones make explicit keys and values of the visible rows.
Routing: sigmoid scores, the best groups of neighbours by the sum of their two best, weights not divided by their sum; the experts'
gated units are bounded.  The head is the embedding table.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Iterator, Optional

import torch

from ..ops import latent as lat
from ..ops import recurrent as rec
from .architecture import ForgetMixArch, FosulixArch, FosulixLayer, LatentAttentionArch
from .windowed import LayerLoopState, LayerWeights, WindowedDecoder, padded


@dataclass
class FosulixLayerWeights(LayerWeights):           # norms: norm1, norm2
    conv: Optional[torch.Tensor] = None            # [taps, W]
    depth: Optional[torch.Tensor] = None           # [layer + 2] fp32
    latent: Optional[lat.LatentWeights] = None
    down_proj: Optional[torch.Tensor] = None       # [query latent | key latent | shared key part, W]
    uq: Optional[torch.Tensor] = None              # [H * dq, query latent]
    forget_spec: Optional[rec.ForgetSpec] = None
    forget: Optional[rec.ForgetWeights] = None
    qfv: Optional[torch.Tensor] = None             # [queries | gates | values, W]

    def tensors(self) -> Iterator[torch.Tensor]:
        yield from super().tensors()
        yield from (self.conv, self.depth)
        if self.latent is not None:
            l = self.latent
            yield from (t for t in (self.down_proj, self.uq, l.ukv, l.q_norm, l.norm) if t is not None)
        else:
            yield from (self.qfv, self.forget.bias, self.forget.lower, self.forget.norm)


class FosulixModel(WindowedDecoder):
    family = "Fosulix"
    arch: FosulixArch

    # ------------------------------------------------------------------- storage
    def _alloc(self) -> None:
        a = self.arch
        if self.device.type == "cuda":
            rows = [l.mixer.cache_row for l in a.layers if not l.recurrent]
            if max(rows, default=0) > lat.MAX_LATENT:
                raise ValueError(f"latent rows of {max(rows)} elements: the attention kernels take at most {lat.MAX_LATENT}")
            if a.taps > rec.MAX_TAPS:
                raise ValueError(f"convolutions of up to {rec.MAX_TAPS} taps, got {a.taps}")
        self.weights = [self._alloc_layer(i, l) for i, l in enumerate(a.layers)]

    def _alloc_layer(self, i: int, l: FosulixLayer) -> FosulixLayerWeights:
        w = FosulixLayerWeights({n: self._z(self.W) for n in ("norm1",) + (("norm2",) if l.moe is not None else ())})
        w.conv, w.depth = self._z(self.arch.taps, self.W), torch.zeros(i + 2, dtype=torch.float32, device=self.device)
        if l.recurrent:
            self._alloc_forget(w, l.mixer)
        else:
            self._alloc_latent(w, l.mixer)
        if l.moe is not None:
            self._alloc_experts(w, l.moe)
        return w

    def _alloc_forget(self, w: FosulixLayerWeights, m: ForgetMixArch) -> None:
        w.forget_spec = s = rec.ForgetSpec(m.heads, m.dim, m.vdim, self.arch.norm_eps)
        lower = torch.ones(s.gate_col, dtype=self.dtype, device=self.device)
        w.forget = rec.ForgetWeights(self._z(s.gate_col), lower, self._z(s.m))
        w.qfv, w.o = self._z(s.proj_cols, self.W), self._z(self.W, m.heads * s.m)

    def _alloc_latent(self, w: FosulixLayerWeights, m: LatentAttentionArch) -> None:
        Q, own = padded(m.q_rank), m.kv_from < 0
        rot = None
        if m.rot_dim:
            freq = torch.tensor(m.rot.inv_freq(), dtype=torch.float64).to(torch.float32).to(self.device)
            rot = lat.Rotary(freq, m.rot_dim, m.rot_start, m.row_rot_start, m.rot.amplitude)
        w.latent = lat.LatentWeights(m.heads, m.dq, m.dv, m.kv_rank, m.scale, self._z(m.row_rot_start) if own else None,
                                     self._z(m.heads * (m.dq + m.dv), m.cache_row), rot, m.window, m.q_rank, self._z(Q))
        w.latent.connect_rotary()
        w.down_proj = self._z(Q + (m.row_rot_start + padded(m.rot_dim) if own else 0), self.W)
        w.uq, w.o = self._z(m.heads * m.dq, Q), self._z(self.W, m.heads * m.dv)

    # ------------------------------------------------------------------- loading
    def _place(self, name: str, t: torch.Tensor) -> bool:
        index, _, sub = name[1:].partition(".")
        if sub == "canon1":
            self._into(self.weights[int(index)].conv[:, :self.arch.width], t.t())
        elif sub == "dwa":
            self._into(self.weights[int(index)].depth, t)
        else:
            return super()._place(name, t)
        return True

    def _place_mixer(self, w: FosulixLayerWeights, sub: str, t: torch.Tensor) -> bool:
        return self._place_forget(w, sub, t) if w.forget is not None else self._place_latent(w, sub, t)

    def _place_forget(self, w: FosulixLayerWeights, sub: str, t: torch.Tensor) -> bool:
        s, width = w.forget_spec, self.arch.width
        H = s.heads
        sections = {"q": (0, s.n, s.dim), "f": (s.gate_col, s.n, s.dim), "v": (s.value_col, s.m, s.vdim)}   # first row, padded and real rows of a head
        if sub in sections:
            first, pad, real = sections[sub]
            self._into(w.qfv[first:first + H * pad].view(H, pad, self.W)[:, :real, :width], t.view(H, real, width))
        elif sub in ("f.b", "lower"):
            self._into((w.forget.bias if sub == "f.b" else w.forget.lower).view(H, s.n)[:, :s.dim], t.view(H, s.dim))
        elif sub == "norm":
            self._into(w.forget.norm[:s.vdim], t)
        elif sub == "o":
            self._into(w.o.view(self.W, H, s.m)[:width, :, :s.vdim], t.view(width, H, s.vdim))
        else:
            return False
        return True

    def _place_latent(self, w: FosulixLayerWeights, sub: str, t: torch.Tensor) -> bool:
        l, width = w.latent, self.arch.width
        H, Q, R = l.heads, l.q_norm.shape[0], l.rank
        if sub == "dq":
            self._into(w.down_proj[:l.q_rank, :width], t)
        elif sub == "dq.norm":
            self._into(l.q_norm[:l.q_rank], t)
        elif sub == "dkv":
            C = l.norm.shape[0]
            self._into(w.down_proj[Q:Q + R, :width], t[:R])
            self._into(w.down_proj[Q + C:Q + C + t.shape[0] - R, :width], t[R:])
        elif sub == "dkv.norm":
            self._into(l.norm[:R], t)
        elif sub == "uq":
            rot = l.rot.dims if l.rot is not None else 0
            per = t.view(H, -1, l.q_rank)
            dim, dst = per.shape[1] - rot, w.uq.view(H, l.dq, Q)
            self._into(dst[:, :dim, :l.q_rank], per[:, :dim])
            if rot:
                self._into(dst[:, l.rot.start:l.rot.start + rot, :l.q_rank], per[:, dim:])
        elif sub == "uk":
            self._into(l.uk.view(H, l.dq, -1)[:, :t.shape[0] // H, :R], t.view(H, -1, R))
        elif sub == "uv":
            self._into(l.uv.view(H, l.dv, -1)[:, :t.shape[0] // H, :R], t.view(H, -1, R))
        elif sub == "o":
            self._into(w.o.view(self.W, H, l.dv)[:width, :, :t.shape[1] // H], t.view(width, H, -1))
        else:
            return False
        return True

    # ---------------------------------------------------------------------- text
    def _state_view(self, st: LayerLoopState, layer: int) -> rec.StateView:
        meta = st.meta
        return rec.StateView(meta.state, layer, meta.state_slots, meta.kv_lens if meta.is_prefill else meta.context_lens,
                             meta.cu_seqlens_q if meta.is_prefill else None)

    def _conv_spec(self, layer: int) -> rec.ConvSpec:
        return rec.ConvSpec(self.arch.taps, self.W, self.arch.carry_start(layer))

    def _layer_input(self, st: LayerLoopState, layer: int) -> dict:
        """What the update behind layer ``layer - 1`` writes: its result, the average, and the normalised rows for the mixer of
        ``layer`` (in a decode step through the convolution already) or for the head."""
        kw = {"history": st.history, "depth": layer, "depth_weight": self.weights[layer - 1].depth if layer else None, "norm_out": st.n}
        if layer == len(self.weights):
            return {**kw, "norm_weight": self.final_norm}
        w = self.weights[layer]
        conv = None if st.meta.is_prefill else rec.ConvStep(w.conv, self._conv_spec(layer), self._state_view(st, layer))
        return {**kw, "norm_weight": w.norms["norm1"], "conv": conv}

    def _embed(self, st: LayerLoopState) -> None:
        st.history = torch.empty((len(self.weights) + 1, *st.x.shape), dtype=torch.float32, device=self.device)
        self._update(st, keep=False, ids=st.ids, table=self.embed, embed_mult=self.arch.embed_scale, **self._layer_input(st, 0))

    def _run_layer(self, st: LayerLoopState, run: int) -> None:
        w, mult = self.weights[run], self.arch.residual_mult
        h = st.n
        if st.meta.is_prefill:
            h = rec.short_conv(st.n, w.conv, self._conv_spec(run), self._state_view(st, run), max_len=st.meta.max_q_len)
        mix = self._project(self._latent(st, w, h, run) if w.latent is not None else self._forget(st, w, h, run), w.o)
        if w.router is not None:
            self._update(st, a=mix, mult=mult, norm_weight=w.norms["norm2"], norm_out=st.n)
            mix = self._experts(st, w, st.n)
        self._update(st, a=mix, mult=mult, **self._layer_input(st, run + 1))

    def _forget(self, st: LayerLoopState, w: FosulixLayerWeights, h: torch.Tensor, run: int) -> torch.Tensor:
        return rec.forget_mix(self._project(h, w.qfv), w.forget_spec, w.forget, self._state_view(st, run))

    def _latent(self, st: LayerLoopState, w: FosulixLayerWeights, h: torch.Tensor, run: int) -> torch.Tensor:
        meta, cache, l, eps, slab = st.meta, st.cache, w.latent, self.arch.norm_eps, self.arch.cache_slab(run)
        q = self._project(lat.latent_prepare(self._project(h, w.down_proj), l, eps, st.positions, meta.slots, cache, slab), w.uq)
        if not meta.is_prefill:
            return lat.latent_attention_absorbed(q, None, None, l, eps, meta.slots, cache, slab, meta.block_tables, meta.context_lens,
                                                 positions=st.positions)
        if self.device.type == "cuda" and self.dtype == torch.bfloat16:
            plan = self._expand_plan(meta, l.window, cache.page)
            if plan.is_cheaper(l, cache.latent(slab).shape[-1], cache.page):
                return lat.latent_attention_windowed(lat.rotate_queries(q, l, st.positions), l, cache, slab, meta.block_tables, meta.kv_lens,
                                                     meta.cu_seqlens_q, meta.max_q_len, plan)
        return lat.latent_attention_absorbed(q, None, None, l, eps, meta.slots, cache, slab, meta.block_tables, meta.kv_lens,
                                             cu_seqlens_q=meta.cu_seqlens_q, max_q_len=meta.max_q_len, positions=st.positions)

    def _expand_plan(self, meta, window: int, page: int) -> lat.ExpandPlan:
        if window not in meta.plans:
            if meta.host_lens is None:
                meta.host_lens = list(zip((meta.cu_seqlens_q[1:] - meta.cu_seqlens_q[:-1]).tolist(), meta.kv_lens.tolist()))
            meta.plans[window] = lat.ExpandPlan.make(meta.host_lens, window, page, meta.block_tables.shape[1], self.device)
        return meta.plans[window]
