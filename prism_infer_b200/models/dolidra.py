"""Dolidra: a looped decoder with windowed attention (differential, or with kept first tokens and head gates), dense and
routed gated feed-forwards, norms on both sides of every sublayer and a per-layer token table, as the engine runs it.

With ``N_w(y)`` a row over its root mean square times ``w``, a layer is

    x += N_1b(O attention(N_1(x)))
    x += N_2b(feed-forward(N_2(x)))            dense (tanh GELU) or top-k experts plus a shared one (SiLU)
    x += N_s(P (gelu_tanh(G x) * table[token, layer]))

The residual ``x`` stays fp32.  Queries, keys, values and head gates are one stacked projection; one kernel adds its bias,
normalises, rotates and stores keys and values in the token's cache row; attention combines maps and gates in its last step;
each ``x +=`` is one kernel that sums the branch (split-K slabs, rows, or weighted expert rows), normalises it, updates ``x``
and hands the next projection its input.  Layers ``loop_start .. loop_stop - 1`` run ``loop_times`` times; every run of a layer
has its own cache slab, of that layer's row width.
"""

from __future__ import annotations

import math
from dataclasses import dataclass, field, replace
from typing import Iterator, Optional

import torch

from .. import ops
from ..ops import latent as lat
from ..ops import window
from .architecture import DolidraLayer
from .windowed import LayerLoopState, LayerWeights, WindowedDecoder, padded


@dataclass
class DolidraLayerWeights(LayerWeights):           # norms: norm1, norm1b, norm2, norm2b, side.norm
    side_gate: Optional[torch.Tensor] = None       # [D, W]
    side_proj: Optional[torch.Tensor] = None       # [W, D]
    lam_dots: dict[str, torch.Tensor] = field(default_factory=dict)  # vectors of the differential weight, while loading

    def tensors(self) -> Iterator[torch.Tensor]:
        yield from super().tensors()
        yield from (self.side_gate, self.side_proj)


class DolidraModel(WindowedDecoder):
    family = "Dolidra"

    # ------------------------------------------------------------------- storage
    def _alloc(self) -> None:
        a = self.arch
        self.D = padded(a.side_dim)
        self.side_table = self._z(a.vocab_size, len(a.layers), self.D)
        self.weights = [self._alloc_layer(l) for l in a.layers]

    def _alloc_layer(self, l: DolidraLayer) -> DolidraLayerWeights:
        W = self.W
        norms = {n: self._z(W) for n in ("norm1", "norm1b", "side.norm") + (("norm2", "norm2b") if l.has_ff else ())}
        w = DolidraLayerWeights(norms, side_gate=self._z(self.D, W), side_proj=self._z(W, self.D))
        self._alloc_attention(w, l.mixer)
        if l.moe is not None:
            self._alloc_experts(w, l.moe)
        elif l.ff:
            w.gate_up, w.down = self._z(2 * padded(l.ff), W), self._z(W, padded(l.ff))
        return w

    def weight_bytes(self) -> int:
        return super().weight_bytes() + self.side_table.numel() * self.side_table.element_size()

    # ------------------------------------------------------------------- loading
    def _place(self, name: str, t: torch.Tensor) -> bool:
        a = self.arch
        index, _, sub = name[1:].partition(".")
        if name == "side.embed":
            self._into(self.side_table[..., :a.side_dim], t.view(t.shape[0], len(a.layers), a.side_dim))
        elif sub == "side.gate":
            self._into(self.weights[int(index)].side_gate[:a.side_dim, :a.width], t)
        elif sub == "side.proj":
            self._into(self.weights[int(index)].side_proj[:a.width, :a.side_dim], t)
        else:
            return super()._place(name, t)
        return True

    def _place_mixer(self, w: DolidraLayerWeights, sub: str, t: torch.Tensor) -> bool:
        if sub in ("lq1", "lk1", "lq2", "lk2"):
            w.lam_dots[sub] = t.detach().double().cpu()
            return True
        return super()._place_mixer(w, sub, t)

    def _loaded(self) -> None:
        for w, l in zip(self.weights, self.arch.layers):
            d = w.lam_dots
            if len(d) == 4:
                lam = math.exp(float(d["lq1"] @ d["lk1"])) - math.exp(float(d["lq2"] @ d["lk2"])) + l.mixer.diff
                w.spec = replace(w.spec, lam=lam)

    # ---------------------------------------------------------------------- text
    def _embed(self, st: LayerLoopState) -> None:
        self._update(st, keep=False, ids=st.ids, table=self.embed, norm_weight=self._input_norm(0), norm_out=st.n)

    def _input_norm(self, run: int) -> torch.Tensor:
        """Weight of the norm in front of layer run ``run``, or of the head."""
        return self.weights[self.runs[run].layer].norms["norm1"] if run < len(self.runs) else self.final_norm

    def _run_layer(self, st: LayerLoopState, run: int) -> None:
        layer = self.runs[run].layer
        w = self.weights[layer]
        mix = self._project(self._attend(st, w, st.n, run), w.o)
        mix.post_norm = w.norms["norm1b"]
        if w.down is None:
            self._update(st, a=mix, raw_out=st.raw)
        else:
            self._update(st, a=mix, norm_weight=w.norms["norm2"], norm_out=st.n)
            ff = self._feed_forward(st, w)
            ff.post_norm = w.norms["norm2b"]
            self._update(st, a=ff, raw_out=st.raw)
        g = window.token_side_gate(self._project(st.raw, w.side_gate), self.side_table, layer, st.ids)
        side = self._project(g, w.side_proj)
        side.post_norm = w.norms["side.norm"]
        self._update(st, a=side, norm_weight=self._input_norm(run + 1), norm_out=st.n)

    def _feed_forward(self, st: LayerLoopState, w: DolidraLayerWeights) -> lat.Branch:
        if w.router is None:
            return self._project(ops.gate_up_glu(st.n, w.gate_up, "gelu_tanh"), w.down)
        return self._experts(st, w, st.n)
