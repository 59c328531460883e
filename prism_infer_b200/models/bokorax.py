"""Bokorax: a decoder that alternates recurrent time mixing with windowed and causal attention, all feed-forwards routed, as
the engine runs it.

With ``N_w(y)`` a row over its root mean square times ``1 + w``, a layer is

    x += N_1(mixer(x))
    x += N_2(experts(x))

so sublayers read the stream itself and only their outputs are normalised.  The mixers:

    wkv            time mixing with a matrix state per head (``ops/recurrent.py``)
    attention      windowed; the values are the keys as projected; norms over the whole query and key rows
    attention_2    causal; norms per head, bounded scores, a sink per head, a gate per head; a layer may read the cached keys
                   and values of an earlier one instead of its own

The residual ``x`` stays fp32 and the recurrent layers blend its rows in 32-bit; attention and experts read its copy in the
compute type.  Cache slabs exist for the layers that have keys of their own, state rows for the recurrent ones.  Routing:
softmax over all outputs, a correction that enters the choice only, the best groups of neighbours, outputs that stand for the
stream's own row, and a shared expert behind a sigmoid per token, whose logit is one more row of the router.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Iterator, Optional

import torch

from ..ops import recurrent as rec
from .architecture import BokoraxLayer, TimeMixArch
from .windowed import LayerLoopState, LayerWeights, WindowedDecoder, padded

MIX_ORDER = "rkvgw"


@dataclass
class BokoraxLayerWeights(LayerWeights):           # norms: norm1, norm2
    mix_spec: Optional[rec.TimeMixSpec] = None
    mix: Optional[rec.TimeMixWeights] = None

    def tensors(self) -> Iterator[torch.Tensor]:
        yield from super().tensors()
        if self.mix is not None:
            m = self.mix
            yield from (m.mu, m.rkvg, m.w1, m.w2, m.w0, m.u, m.norm)


class BokoraxModel(WindowedDecoder):
    family = "Bokorax"

    # ------------------------------------------------------------------- storage
    def _alloc(self) -> None:
        self.weights = [self._alloc_layer(l) for l in self.arch.layers]

    def _alloc_layer(self, l: BokoraxLayer) -> BokoraxLayerWeights:
        w = BokoraxLayerWeights({n: self._z(self.W) for n in ("norm1",) + (("norm2",) if l.moe is not None else ())})
        if l.recurrent:
            self._alloc_time_mix(w, l.mixer)
        else:
            self._alloc_attention(w, l.mixer)
        if l.moe is not None:
            self._alloc_experts(w, l.moe)
        return w

    def _alloc_time_mix(self, w: BokoraxLayerWeights, m: TimeMixArch) -> None:
        w.mix_spec = s = rec.TimeMixSpec(m.heads, m.dim, padded(m.decay_rank), self.W, self.arch.norm_eps)
        w.mix = rec.TimeMixWeights(mu=self._z(5, self.W), rkvg=self._z(4, s.cols, self.W), w1=self._z(s.rank, self.W),
                                   w2=self._z(s.cols, s.rank), w0=self._z(s.cols), u=self._z(s.cols), norm=self._z(s.cols))
        w.o = self._z(self.W, s.cols)

    # ------------------------------------------------------------------- loading
    def _place_mixer(self, w: BokoraxLayerWeights, sub: str, t: torch.Tensor) -> bool:
        return self._place_time_mix(w, sub, t) if w.mix is not None else self._place_attention(w, sub, t)

    def _place_time_mix(self, w: BokoraxLayerWeights, sub: str, t: torch.Tensor) -> bool:
        s, m, width = w.mix_spec, w.mix, self.arch.width
        H, d, rank = s.heads, s.dim, t.shape[-1]

        def heads(dst: torch.Tensor) -> torch.Tensor:
            """The real rows of a tensor with a row (or an element) per padded channel."""
            return dst.view(H, s.n, *dst.shape[1:])[:, :d]

        if sub.startswith("mu."):
            self._into(m.mu[MIX_ORDER.index(sub[3:]), :width], t)
        elif sub in ("r", "k", "v", "g"):
            self._into(heads(m.rkvg[MIX_ORDER.index(sub)])[..., :width], t.view(H, d, width))
        elif sub == "w1":
            self._into(m.w1[:t.shape[0], :width], t)
        elif sub == "w2":
            self._into(heads(m.w2)[..., :rank], t.view(H, d, rank))
        elif sub in ("w0", "u", "norm"):
            self._into(heads(getattr(m, sub)), t.view(H, d))
        elif sub == "o":
            self._into(w.o.view(self.W, H, s.n)[:width, :, :d], t.view(width, H, d))
        else:
            return False
        return True

    # ---------------------------------------------------------------------- text
    def _hand_on(self, st: LayerLoopState, layer: int) -> dict:
        """What an update writes for the mixer of ``layer`` (a recurrent one reads the stream itself), or for the head behind the
        last one."""
        if layer == len(self.weights):
            return {"norm_weight": self.final_norm, "norm_out": st.n}
        return {} if self.weights[layer].mix is not None else {"raw_out": st.raw}

    def _embed(self, st: LayerLoopState) -> None:
        self._update(st, keep=False, ids=st.ids, table=self.embed, embed_mult=self.arch.embed_scale, **self._hand_on(st, 0))

    def _run_layer(self, st: LayerLoopState, run: int) -> None:
        w = self.weights[run]
        mix = self._project(self._time_mix(st, w, run) if w.mix is not None else self._attend(st, w, st.raw, self.arch.cache_slab(run)), w.o)
        mix.post_norm = w.norms["norm1"]
        if w.router is None:
            self._update(st, a=mix, norm_offset=1.0, **self._hand_on(st, run + 1))
            return
        self._update(st, a=mix, norm_offset=1.0, raw_out=st.raw)
        ff = self._experts(st, w, st.raw)
        ff.post_norm = w.norms["norm2"]
        self._update(st, a=ff, norm_offset=1.0, **self._hand_on(st, run + 1))

    def _time_mix(self, st: LayerLoopState, w: BokoraxLayerWeights, run: int) -> torch.Tensor:
        meta = st.meta
        view = rec.StateView(meta.state, self.arch.state_slab(run), meta.state_slots, meta.kv_lens if meta.is_prefill else meta.context_lens,
                             meta.cu_seqlens_q if meta.is_prefill else None)
        return rec.time_mix(st.x, w.mix_spec, w.mix, view)
