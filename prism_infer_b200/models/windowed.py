"""What the families with attention over single-row caches and routed experts share: padded packed weights of a
layer, their loading, the layer loop's skeleton, projections, attention, experts, logits and sampling.

Inner dimensions are zero-padded at load time to multiples of 16; padding stays zero through every operation and norms count
real columns only.  A shared expert is stored as one or more experts of the routed width that every token uses.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Iterable, Iterator, Optional

import torch

from .. import ops
from ..ops import latent as lat
from ..ops import moe, window
from .architecture import LayerRun, MixtureArch, WindowAttentionArch
from .common import AttnMeta, TPComm


def padded(n: int, to: int = 16) -> int:
    return -(-n // to) * to


@dataclass
class LayerWeights:
    norms: dict[str, torch.Tensor] = field(default_factory=dict)   # [W] each
    spec: Optional[window.WindowSpec] = None
    qkv: Optional[torch.Tensor] = None      # [proj_cols, W]
    attn: Optional[window.WindowWeights] = None
    o: Optional[torch.Tensor] = None        # [W, H * dv]
    gate_up: Optional[torch.Tensor] = None  # dense [2 F, W] or experts [E, 2 F, W]
    down: Optional[torch.Tensor] = None     # dense [W, F] or experts [E, W, F]
    router: Optional[torch.Tensor] = None   # [outputs, W], with one more row for the shared expert's gate
    top: int = 0                            # routed experts of a token
    always: int = 0                         # experts after the routed ones that every token uses
    experts: int = 0
    scored: Optional[moe.Scored] = None
    limit: float = 0.0                      # bound of the experts' gated units (0: SiLU units)

    def tensors(self) -> Iterator[torch.Tensor]:
        a = self.attn or window.WindowWeights()
        yield from (t for t in (self.qkv, a.bias, a.q_norm, a.k_norm, a.sink, self.o, self.gate_up, self.down, self.router,
                                *self.norms.values()) if t is not None)


@dataclass
class LayerLoopState:
    """What the layer loop carries from one layer run to the next."""

    meta: AttnMeta
    cache: "ops.KVCache"
    ids: torch.Tensor                      # [T] token ids
    positions: torch.Tensor                # [T] int32
    x: torch.Tensor                        # [T, W] fp32 residual stream
    n: torch.Tensor                        # [T, W] normalised rows: input of the next projection
    raw: torch.Tensor                      # [T, W] the stream in the compute type
    next_layer: int = 0
    history: Optional[torch.Tensor] = None # [n, T, W] fp32 results of the layers so far, where a design reads them again


class WindowedDecoder:
    family = ""

    def __init__(self, arch, *, device, dtype: torch.dtype, comm: TPComm | None = None) -> None:
        self.arch = arch
        self.device = torch.device(device)
        self.dtype = dtype
        self.comm = comm or TPComm()
        if self.comm.size != 1:
            raise ValueError(f"the {self.family} family runs on one rank")
        self.W = padded(arch.width)
        self.runs: tuple[LayerRun, ...] = arch.layer_runs()
        self.layers = self.runs            # what the layer-quantum prefill counts
        self.sampled_logits: Optional[torch.Tensor] = None
        self.keep_logits = False
        self._head_sections = lat.Sections([(arch.vocab_size, getattr(arch, "logit_scale", 1.0), None)])
        self.embed, self.final_norm = self._z(arch.vocab_size, self.W), self._z(self.W)
        self.head = self.embed if getattr(arch, "tied_head", False) else self._z(arch.vocab_size, self.W)
        self._alloc()

    # ------------------------------------------------------------------- storage
    def _z(self, *shape: int) -> torch.Tensor:
        return torch.zeros(shape, dtype=self.dtype, device=self.device)

    def _alloc(self) -> None:
        raise NotImplementedError

    def _alloc_attention(self, w: LayerWeights, m: WindowAttentionArch) -> None:
        w.spec = s = window.WindowSpec(
            heads=m.heads, kv_heads=m.kv_heads, maps=m.maps, dim=m.dim, vdim=m.vdim, rot_dims=m.rot.dims, scale=m.scale, window=m.window,
            keep_first=m.keep_first, gate=m.gate, eps=self.arch.norm_eps, gain=1.0 - m.diff if m.maps == 2 else 1.0,
            head_norm=m.head_norm, tied=m.tied_values, shared=m.kv_from >= 0, softcap=m.softcap)
        norms = {}
        if m.qk_norm:
            norms["q_norm"] = self._z(s.dq if m.head_norm else s.q_cols)
            if not s.shared:
                norms["k_norm"] = self._z(s.dq if m.head_norm else s.k_cols)
        w.attn = window.WindowWeights(
            bias=self._z(s.proj_cols) if m.bias else None, inv_freq=torch.tensor(m.rot.inv_freq(), dtype=torch.float64).to(torch.float32).to(self.device),
            sink=torch.zeros(m.heads, dtype=torch.float32, device=self.device) if m.sink else None, **norms)
        w.qkv, w.o = self._z(s.proj_cols, self.W), self._z(self.W, m.heads * s.dv)

    def _alloc_experts(self, w: LayerWeights, m: MixtureArch) -> None:
        F, E = padded(m.ff), m.experts
        w.top, w.always, w.experts, w.limit = m.top, -(-m.shared_ff // F), E, m.limit
        w.gate_up, w.down = self._z(E + w.always, 2 * F, self.W), self._z(E + w.always, self.W, F)
        w.router = self._z(m.outputs + m.shared_gate, self.W)
        if m.scored:
            w.scored = moe.Scored(torch.zeros(m.outputs, dtype=torch.float32, device=self.device), m.identity, m.groups, m.groups_kept, m.scale,
                                  m.shared_gate, m.sigmoid, 2 if m.sigmoid else 1)

    def weight_bytes(self) -> int:
        tensors = [self.embed, self.final_norm] + ([] if self.head is self.embed else [self.head]) + [t for w in self.weights for t in w.tensors()]
        return sum(t.numel() * t.element_size() for t in tensors)

    # ------------------------------------------------------------------- loading
    @staticmethod
    def _into(dst: torch.Tensor, src: torch.Tensor) -> None:
        dst.copy_(src.to(device=dst.device, dtype=dst.dtype))

    def _place(self, name: str, t: torch.Tensor) -> bool:
        """Copy one checkpoint tensor into its padded place; False for a tensor the model has no use for."""
        width = self.arch.width
        if name in ("embed", "head"):
            self._into(getattr(self, name)[:, :width], t)
        elif name == "final.norm":
            self._into(self.final_norm[:width], t)
        else:
            index, _, sub = name[1:].partition(".")
            w, l = self.weights[int(index)], self.arch.layers[int(index)]
            if sub in w.norms:
                self._into(w.norms[sub][:width], t)
            elif sub.startswith("mix."):
                return self._place_mixer(w, sub[4:], t)
            elif sub.startswith("mlp."):
                return self._place_ff(w, l, sub[4:], t)
            else:
                return False
        return True

    def _place_mixer(self, w: LayerWeights, sub: str, t: torch.Tensor) -> bool:
        return self._place_attention(w, sub, t)

    def _place_attention(self, w: LayerWeights, sub: str, t: torch.Tensor) -> bool:
        s, width = w.spec, self.arch.width
        # section -> (first row, heads in it, padded and real rows of one)
        sections = {"q": (0, s.heads * s.maps, s.dq, s.dim), "k": (s.q_cols, s.kv_heads * s.maps, s.dq, s.dim),
                    "v": (s.q_cols + s.k_cols, s.kv_heads, s.dv, s.vdim)}
        part, _, kind = sub.partition(".")
        if part in sections:
            first, n, pad, real = sections[part]
            if kind == "":
                self._into(w.qkv[first:first + n * pad].view(n, pad, self.W)[:, :real, :width], t.view(n, real, width))
            elif kind == "b":
                self._into(w.attn.bias[first:first + n * pad].view(n, pad)[:, :real], t.view(n, real))
            else:
                if s.head_norm:
                    n = 1
                self._into((w.attn.q_norm if part == "q" else w.attn.k_norm).view(n, pad)[:, :real], t.view(n, real))
        elif sub == "g":
            self._into(w.qkv[s.gate_row:s.gate_row + s.heads, :width], t)
        elif sub == "o":
            self._into(w.o.view(self.W, s.heads, s.dv)[:width, :, :s.vdim], t.view(width, s.heads, s.vdim))
        elif sub == "sink":
            self._into(w.attn.sink, t)
        else:
            return False
        return True

    def _place_ff(self, w: LayerWeights, l, sub: str, t: torch.Tensor) -> bool:
        width = self.arch.width
        if sub == "router":
            self._into(w.router[:t.shape[0], :width], t)
        elif sub == "correction":
            self._into(w.scored.correction, t)
        elif sub == "shared.sg":
            self._into(w.router[-1:, :width], t)
        else:
            owner, _, kind = sub.rpartition(".")
            if l.moe is None:
                self._place_glu(w.gate_up, w.down, kind, t)
            elif owner == "shared":            # blocks of the routed width
                F = w.down.shape[2]
                for k, lo in enumerate(range(0, l.moe.shared_ff, F)):
                    part = t[:, lo:lo + F] if kind == "down" else t[lo:lo + F]
                    self._place_glu(w.gate_up[l.moe.experts + k], w.down[l.moe.experts + k], kind, part)
            else:
                self._place_glu(w.gate_up[int(owner[1:])], w.down[int(owner[1:])], kind, t)
        return True

    def _place_glu(self, gate_up: torch.Tensor, down: torch.Tensor, kind: str, t: torch.Tensor) -> None:
        width = self.arch.width
        if kind == "down":
            self._into(down[:width, :t.shape[1]], t)
        else:
            first = 0 if kind == "gate" else down.shape[1]
            self._into(gate_up[first:first + t.shape[0], :width], t)

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
        self._loaded()

    def _loaded(self) -> None:
        """What follows from the loaded tensors."""

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
            raise ValueError(f"the {self.family} family takes text only")
        T = input_ids.shape[0]
        x = torch.empty((T, self.W), dtype=torch.float32, device=self.device)
        n, raw = (torch.empty((T, self.W), dtype=self.dtype, device=self.device) for _ in range(2))
        st = LayerLoopState(meta, cache, input_ids, positions[0], x, n, raw)
        self._embed(st)
        return st

    def _embed(self, st: LayerLoopState) -> None:
        raise NotImplementedError

    def _run_layer(self, st: LayerLoopState, run: int) -> None:
        raise NotImplementedError

    def _update(self, st: LayerLoopState, *, keep: bool = True, **kw) -> None:
        lat.stream_update(st.x, self.arch.width, self.arch.norm_eps, keep=keep, **kw)

    @torch.no_grad()
    def advance_layers(self, st: LayerLoopState, max_layers: int) -> bool:
        """Run up to ``max_layers`` more layer runs; True once all have run."""
        stop = min(len(self.runs), st.next_layer + max(0, int(max_layers)))
        for i in range(st.next_layer, stop):
            self._run_layer(st, i)
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

    def _attend(self, st: LayerLoopState, w: LayerWeights, h: torch.Tensor, slab: int) -> torch.Tensor:
        meta, cache = st.meta, st.cache
        q, gate = window.qkv_prepare(self._project(h, w.qkv), w.spec, w.attn, st.positions, meta.slots, cache, slab)
        if not meta.is_prefill:
            return window.window_attention(q, w.spec, gate, cache, slab, meta.block_tables, meta.context_lens, sink=w.attn.sink)
        return window.window_attention(q, w.spec, gate, cache, slab, meta.block_tables, meta.kv_lens, cu_seqlens_q=meta.cu_seqlens_q,
                                       max_q_len=meta.max_q_len, sink=w.attn.sink)

    def _experts(self, st: LayerLoopState, w: LayerWeights, h: torch.Tensor) -> lat.Branch:
        routing = moe.route(lat.Branch(slabs=lat.linear_slabs(h, w.router)), w.top, w.experts, w.always, st.meta.slots,
                            f32=self.dtype == torch.float32, scored=w.scored)
        return moe.expert_ffn(h, routing, w.gate_up, w.down, "bounded" if w.limit > 0.0 else "silu", w.limit)

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
