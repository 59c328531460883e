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

Inner dimensions are zero-padded at load time to multiples of 16; padding stays zero through every operation and norms count
real columns only.  A shared expert is stored as one or more experts of the routed width that every token uses.
"""

from __future__ import annotations

import math
from dataclasses import dataclass, field, replace
from typing import Iterable, Iterator, Optional

import torch

from .. import ops
from ..ops import latent as lat
from ..ops import moe, window
from .architecture import DolidraArch, DolidraLayer, LayerRun
from .common import AttnMeta, TPComm


def _up(n: int, to: int = 16) -> int:
    return -(-n // to) * to


@dataclass
class DolidraLayerWeights:
    spec: window.WindowSpec
    qkv: torch.Tensor                      # [proj_cols, W]
    attn: window.WindowWeights
    o: torch.Tensor                        # [W, H * dv]
    norms: dict[str, torch.Tensor]         # norm1, norm1b, norm2, norm2b, side: [W]
    side_gate: torch.Tensor                # [D, W]
    side_proj: torch.Tensor                # [W, D]
    gate_up: Optional[torch.Tensor] = None  # dense [2 F, W] or experts [E, 2 F, W]
    down: Optional[torch.Tensor] = None     # dense [W, F] or experts [E, W, F]
    router: Optional[torch.Tensor] = None   # [experts, W]
    top: int = 0                            # routed experts of a token
    always: int = 0                         # experts after the routed ones that every token uses
    lam_dots: dict[str, torch.Tensor] = field(default_factory=dict)  # vectors of the differential weight, while loading

    def tensors(self) -> Iterator[torch.Tensor]:
        a = self.attn
        yield from (t for t in (self.qkv, a.bias, a.q_norm, a.k_norm, self.o, self.side_gate, self.side_proj, self.gate_up, self.down,
                                self.router, *self.norms.values()) if t is not None)


@dataclass
class LayerLoopState:
    """What the layer loop carries from one layer run to the next."""

    meta: AttnMeta
    cache: "ops.KVCache"
    ids: torch.Tensor                      # [T] token ids
    positions: torch.Tensor                # [T] int32
    x: torch.Tensor                        # [T, W] fp32 residual stream
    n: torch.Tensor                        # [T, W] normalised rows: input of the next projection
    raw: torch.Tensor                      # [T, W] the stream in the compute type: input of the side gate
    next_layer: int = 0


class DolidraModel:
    def __init__(self, arch: DolidraArch, *, device, dtype: torch.dtype, comm: TPComm | None = None) -> None:
        self.arch = arch
        self.device = torch.device(device)
        self.dtype = dtype
        self.comm = comm or TPComm()
        if self.comm.size != 1:
            raise ValueError("the Dolidra family runs on one rank")
        self.W = _up(arch.width)
        self.D = _up(arch.side_dim)
        self.runs: tuple[LayerRun, ...] = arch.layer_runs()
        self.layers = self.runs            # what the layer-quantum prefill counts
        self.sampled_logits: Optional[torch.Tensor] = None
        self.keep_logits = False
        self._head_sections = lat.Sections([(arch.vocab_size, 1.0, None)])
        self._alloc()

    # ------------------------------------------------------------------- storage
    def _z(self, *shape: int) -> torch.Tensor:
        return torch.zeros(shape, dtype=self.dtype, device=self.device)

    def _alloc(self) -> None:
        a = self.arch
        self.embed, self.head, self.final_norm = self._z(a.vocab_size, self.W), self._z(a.vocab_size, self.W), self._z(self.W)
        self.side_table = self._z(a.vocab_size, len(a.layers), self.D)
        self.weights = [self._alloc_layer(l) for l in a.layers]

    def _alloc_layer(self, l: DolidraLayer) -> DolidraLayerWeights:
        m, W = l.mixer, self.W
        spec = window.WindowSpec(heads=m.heads, kv_heads=m.kv_heads, maps=m.maps, dim=m.dim, vdim=m.vdim, rot_dims=m.rot.dims, scale=m.scale,
                                 window=m.window, keep_first=m.keep_first, gate=m.gate, eps=self.arch.norm_eps,
                                 gain=1.0 - m.diff if m.maps == 2 else 1.0)
        attn = window.WindowWeights(
            bias=self._z(spec.proj_cols) if m.bias else None, q_norm=self._z(spec.q_cols) if m.qk_norm else None,
            k_norm=self._z(spec.k_cols) if m.qk_norm else None,
            inv_freq=torch.tensor(m.rot.inv_freq(), dtype=torch.float64).to(torch.float32).to(self.device))
        norms = {n: self._z(W) for n in ("norm1", "norm1b", "side") + (("norm2", "norm2b") if l.has_ff else ())}
        w = DolidraLayerWeights(spec, self._z(spec.proj_cols, W), attn, self._z(W, m.heads * spec.dv), norms, self._z(self.D, W),
                                self._z(W, self.D))
        if l.moe is not None:
            F, E = _up(l.moe.ff), l.moe.experts
            w.top, w.always = l.moe.top, -(-l.moe.shared_ff // F)
            w.gate_up, w.down, w.router = self._z(E + w.always, 2 * F, W), self._z(E + w.always, W, F), self._z(E, W)
        elif l.ff:
            w.gate_up, w.down = self._z(2 * _up(l.ff), W), self._z(W, _up(l.ff))
        return w

    def weight_bytes(self) -> int:
        tensors = [self.embed, self.head, self.final_norm, self.side_table] + [t for w in self.weights for t in w.tensors()]
        return sum(t.numel() * t.element_size() for t in tensors)

    # ------------------------------------------------------------------- loading
    def _place(self, name: str, t: torch.Tensor) -> bool:
        """Copy one checkpoint tensor into its padded place; False for a tensor the model has no use for."""
        width = self.arch.width

        def into(dst: torch.Tensor, src: torch.Tensor) -> None:
            dst.copy_(src.to(device=self.device, dtype=self.dtype))

        if name in ("embed", "head"):
            into(getattr(self, name)[:, :width], t)
        elif name == "final.norm":
            into(self.final_norm[:width], t)
        elif name == "side.embed":
            into(self.side_table[..., :self.arch.side_dim], t.view(t.shape[0], len(self.arch.layers), self.arch.side_dim))
        else:
            index, _, sub = name[1:].partition(".")
            w, l = self.weights[int(index)], self.arch.layers[int(index)]
            if sub in ("norm1", "norm1b", "norm2", "norm2b"):
                into(w.norms[sub][:width], t)
            elif sub == "side.norm":
                into(w.norms["side"][:width], t)
            elif sub == "side.gate":
                into(w.side_gate[:self.arch.side_dim, :width], t)
            elif sub == "side.proj":
                into(w.side_proj[:width, :self.arch.side_dim], t)
            elif sub.startswith("mix."):
                return self._place_mixer(w, sub[4:], t, into)
            elif sub.startswith("mlp."):
                return self._place_ff(w, l, sub[4:], t, into)
            else:
                return False
        return True

    def _place_mixer(self, w: DolidraLayerWeights, sub: str, t: torch.Tensor, into) -> bool:
        s, width = w.spec, self.arch.width
        # section -> (first row, heads in it, padded and real rows of one)
        sections = {"q": (0, s.heads * s.maps, s.dq, s.dim), "k": (s.q_cols, s.kv_heads * s.maps, s.dq, s.dim),
                    "v": (s.q_cols + s.k_cols, s.kv_heads, s.dv, s.vdim)}
        part, _, kind = sub.partition(".")
        if part in sections:
            first, n, padded, real = sections[part]
            if kind == "":
                into(w.qkv[first:first + n * padded].view(n, padded, self.W)[:, :real, :width], t.view(n, real, width))
            elif kind == "b":
                into(w.attn.bias[first:first + n * padded].view(n, padded)[:, :real], t.view(n, real))
            else:
                into((w.attn.q_norm if part == "q" else w.attn.k_norm).view(n, padded)[:, :real], t.view(n, real))
        elif sub == "g":
            first = s.q_cols + s.k_cols + s.v_cols
            into(w.qkv[first:first + s.heads, :width], t)
        elif sub == "o":
            into(w.o.view(self.W, s.heads, s.dv)[:width, :, :s.vdim], t.view(width, s.heads, s.vdim))
        elif sub in ("lq1", "lk1", "lq2", "lk2"):
            w.lam_dots[sub] = t.detach().double().cpu()
        else:
            return False
        return True

    def _place_ff(self, w: DolidraLayerWeights, l: DolidraLayer, sub: str, t: torch.Tensor, into) -> bool:
        width = self.arch.width
        if sub == "router":
            into(w.router[:, :width], t)
            return True
        owner, _, kind = sub.rpartition(".")
        if l.moe is None:
            self._place_glu(w.gate_up, w.down, kind, t, into)
        elif owner == "shared":            # blocks of the routed width
            F = w.down.shape[2]
            for k, lo in enumerate(range(0, l.moe.shared_ff, F)):
                part = t[:, lo:lo + F] if kind == "down" else t[lo:lo + F]
                self._place_glu(w.gate_up[l.moe.experts + k], w.down[l.moe.experts + k], kind, part, into)
        else:
            self._place_glu(w.gate_up[int(owner[1:])], w.down[int(owner[1:])], kind, t, into)
        return True

    def _place_glu(self, gate_up: torch.Tensor, down: torch.Tensor, kind: str, t: torch.Tensor, into) -> None:
        width = self.arch.width
        if kind == "down":
            into(down[:width, :t.shape[1]], t)
        else:
            first = 0 if kind == "gate" else down.shape[1]
            into(gate_up[first:first + t.shape[0], :width], t)

    def load(self, tensors: Iterable[tuple[str, torch.Tensor]], *, strict: bool = True) -> None:
        """Copy checkpoint tensors into the packed, padded storage."""
        expected = self.arch.weight_shapes()
        seen: set[str] = set()
        for name, tensor in tensors:
            if name not in expected:
                continue
            if tuple(tensor.shape) != expected[name]:
                raise ValueError(f"{name}: checkpoint shape {tuple(tensor.shape)}, the configuration asks for {expected[name]}")
            if not self._place(name, tensor):
                raise KeyError(f"no destination for checkpoint tensor {name}")
            seen.add(name)
        missing = set(expected) - seen
        if strict and missing:
            raise KeyError(f"checkpoint is missing {len(missing)} tensors, e.g. {sorted(missing)[:3]}")
        for w, l in zip(self.weights, self.arch.layers):
            d = w.lam_dots
            if len(d) == 4:
                lam = math.exp(float(d["lq1"] @ d["lk1"])) - math.exp(float(d["lq2"] @ d["lk2"])) + l.mixer.diff
                w.spec = replace(w.spec, lam=lam)

    # ---------------------------------------------------------------------- text
    @torch.no_grad()
    def forward(self, input_ids: torch.Tensor, positions: torch.Tensor, meta: AttnMeta, cache: "ops.KVCache", *,
                visual=None, vis_index=None, deepstack=None) -> torch.Tensor:
        """Rows ``[T, W]`` after the final norm."""
        state = self.begin_layers(input_ids, positions, meta, cache, visual=visual, vis_index=vis_index, deepstack=deepstack)
        self.advance_layers(state, len(self.runs))
        return self.finish_layers(state)

    @torch.no_grad()
    def begin_layers(self, input_ids: torch.Tensor, positions: torch.Tensor, meta: AttnMeta, cache: "ops.KVCache", *,
                     visual=None, vis_index=None, deepstack=None) -> LayerLoopState:
        if visual is not None or deepstack:
            raise ValueError("the Dolidra family takes text only")
        T = input_ids.shape[0]
        x = torch.empty((T, self.W), dtype=torch.float32, device=self.device)
        n, raw = (torch.empty((T, self.W), dtype=self.dtype, device=self.device) for _ in range(2))
        st = LayerLoopState(meta, cache, input_ids, positions[0], x, n, raw)
        self._update(st, keep=False, ids=input_ids, table=self.embed, norm_weight=self._input_norm(0), norm_out=n)
        return st

    def _input_norm(self, run: int) -> torch.Tensor:
        """Weight of the norm in front of layer run ``run``, or of the head."""
        return self.weights[self.runs[run].layer].norms["norm1"] if run < len(self.runs) else self.final_norm

    def _update(self, st: LayerLoopState, *, keep: bool = True, **kw) -> None:
        lat.stream_update(st.x, self.arch.width, self.arch.norm_eps, keep=keep, **kw)

    @torch.no_grad()
    def advance_layers(self, st: LayerLoopState, max_layers: int) -> bool:
        """Run up to ``max_layers`` more layer runs; True once all have run."""
        stop = min(len(self.runs), st.next_layer + max(0, int(max_layers)))
        for i in range(st.next_layer, stop):
            layer = self.runs[i].layer
            w = self.weights[layer]
            mix = self._project(self._attend(st, w, i), w.o)
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
            side.post_norm = w.norms["side"]
            self._update(st, a=side, norm_weight=self._input_norm(i + 1), norm_out=st.n)
        st.next_layer = stop
        return stop == len(self.runs)

    @torch.no_grad()
    def finish_layers(self, st: LayerLoopState) -> torch.Tensor:
        if st.next_layer != len(self.runs):
            raise RuntimeError(f"finish_layers after {st.next_layer} of {len(self.runs)} layer runs")
        return st.n

    def _project(self, x: torch.Tensor, w: torch.Tensor) -> lat.Branch:
        """A projection whose sum the next kernel forms: split-K slabs for up to a few hundred tokens, rows for long prompts."""
        if self.device.type == "cuda" and (self.dtype == torch.float32 or ops.narrow_splits(w.shape[0], w.shape[1], x.shape[0]) > 1):
            return lat.Branch(slabs=lat.linear_slabs(x, w))
        dense, partials, _ = self.comm.row_parallel(x, w)
        return lat.Branch(slabs=partials, rows=dense)

    def _attend(self, st: LayerLoopState, w: DolidraLayerWeights, slab: int) -> torch.Tensor:
        meta, cache = st.meta, st.cache
        q, gate = window.qkv_prepare(self._project(st.n, w.qkv), w.spec, w.attn, st.positions, meta.slots, cache, slab)
        if not meta.is_prefill:
            return window.window_attention(q, w.spec, gate, cache, slab, meta.block_tables, meta.context_lens)
        return window.window_attention(q, w.spec, gate, cache, slab, meta.block_tables, meta.kv_lens, cu_seqlens_q=meta.cu_seqlens_q,
                                       max_q_len=meta.max_q_len)

    def _feed_forward(self, st: LayerLoopState, w: DolidraLayerWeights) -> lat.Branch:
        if w.router is None:
            return self._project(ops.gate_up_glu(st.n, w.gate_up, "gelu_tanh"), w.down)
        routing = moe.route(lat.Branch(slabs=lat.linear_slabs(st.n, w.router)), w.top, w.router.shape[0], w.always, st.meta.slots,
                            f32=self.dtype == torch.float32)
        return moe.expert_ffn(st.n, routing, w.gate_up, w.down, "silu")

    @torch.no_grad()
    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        """fp32 logits ``[B, vocab]``."""
        return lat.linear_sections(hidden, self.head, self._head_sections, out_f32=True)

    @torch.no_grad()
    def sample(self, hidden: torch.Tensor, temperature: Optional[torch.Tensor], *, seed: int = 0,
               step: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        logits = self.sampled_logits = self.logits(hidden)
        if self.keep_logits:
            self.last_logits = logits.clone()
        return ops.sample(logits, temperature, seed=seed, step=step, out=out)
