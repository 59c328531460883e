"""Poralorn: a looped, parallel, gated decoder with latent attention, as the engine runs it.

With ``n`` the residual row over its root mean square, a layer is

    p  = act(alpha * (n W^T) + b)                   one stacked projection: query, latent, output gate, residual gate,
                                                    feed-forward input and its residual gate; the two norms of the
                                                    layer differ by a scalar gain, which is the section's ``alpha``
    x += mult * (sigmoid-gate1 * (O a) + sigmoid-gate2 * (D gelu))

where ``a`` is latent attention (``ops/latent.py``: absorbed over the paged latents for decode steps and short
portions, expanded to keys and values on the tcgen05 kernel for whole prompts).  The residual ``x`` stays fp32; one
kernel adds both branches, normalises and hands the next projection its input.  Layers ``loop_start ..
loop_stop - 1`` run ``loop_times`` times; every run of a layer has its own cache slab, and each pass begins with a
projection of the stream beside the embedding plus a learned vector.

All inner dimensions are zero-padded at load time to what the kernels want (rows of a stacked section and the
width to 16, heads to 8, latents to 64); padding stays zero through every operation and the norms count real
columns only.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Iterable, Iterator, Optional

import torch

from .. import ops
from ..ops import latent as lat
from .architecture import LayerRun, PoralornArch
from .common import AttnMeta, TPComm


def _up(n: int, to: int) -> int:
    return -(-n // to) * to


@dataclass
class PoralornLayerWeights:
    proj: torch.Tensor                     # stacked projections [rows, W]
    bias: torch.Tensor                     # [rows]
    cols: dict[str, tuple[int, int]]       # section -> (first row, rows); every section starts at a multiple of 16
    latent: lat.LatentWeights
    o: torch.Tensor                        # [W, H * dv]
    down: Optional[torch.Tensor]           # [W, F]
    gain1: float = 1.0
    gain2: float = 1.0
    sections: Optional[lat.Sections] = None

    def part(self, p: torch.Tensor, name: str) -> torch.Tensor:
        lo, n = self.cols[name]
        return p[:, lo:lo + n]


@dataclass
class LayerLoopState:
    """What the layer loop carries from one layer run to the next."""

    meta: AttnMeta
    cache: "ops.KVCache"
    x: torch.Tensor                        # [T, W] fp32 residual stream
    n: torch.Tensor                        # [T, W] its normalised rows
    pair: Optional[torch.Tensor]           # [T, 2 W] stream and embedding: input of the loop projection
    next_layer: int = 0


class PoralornModel:
    def __init__(self, arch: PoralornArch, *, device, dtype: torch.dtype, comm: TPComm | None = None) -> None:
        self.arch = arch
        self.device = torch.device(device)
        self.dtype = dtype
        self.comm = comm or TPComm()
        if self.comm.size != 1:
            raise ValueError("the Poralorn family runs on one rank")
        self.W = _up(arch.width, 16)
        self.Rc = arch.latent_row
        self.runs: tuple[LayerRun, ...] = arch.layer_runs()
        self.layers = self.runs            # what the layer-quantum prefill counts
        self.sampled_logits: Optional[torch.Tensor] = None
        self.keep_logits = False
        if self.device.type == "cuda" and self.Rc > lat.MAX_LATENT:
            raise ValueError(f"latent rows of {self.Rc} elements: the attention kernels take at most {lat.MAX_LATENT}")
        self._alloc()

    # ------------------------------------------------------------------- storage
    def _z(self, *shape: int) -> torch.Tensor:
        return torch.zeros(shape, dtype=self.dtype, device=self.device)

    def _alloc(self) -> None:
        a = self.arch
        self.embed = self._z(a.vocab_size, self.W)
        self.head = self._z(a.vocab_size, self.W)
        self.loop_in = self._z(self.W, 2 * self.W) if a.has_loop else None
        self.loop_step = self._z(a.loop_times, self.W) if a.has_loop else None
        self.final_gain = 1.0
        self.head_sections: Optional[lat.Sections] = None
        self.weights: list[PoralornLayerWeights] = []
        for l in a.layers:
            m = l.mixer
            dq, dv = _up(m.dim, 8), _up(m.vdim, 8)
            if max(dq, dv) <= lat.FLASH_MAX_HEAD:  # one width for both: the tcgen05 kernel takes square heads
                dq = dv = max(dq, dv)
            rows = {"q": m.heads * dq, "dkv": m.kv_rank, "g": m.heads * dv, "rg1": self.W}
            if l.ff:
                rows.update({"up": _up(l.ff, 16), "rg2": self.W})
            cols, total = {}, 0
            for name, n in rows.items():
                cols[name] = (total, n)
                total += _up(n, 16)
            latent = lat.LatentWeights(m.heads, dq, dv, m.kv_rank, m.scale, self._z(m.kv_rank), self._z(m.heads * (dq + dv), self.Rc))
            self.weights.append(PoralornLayerWeights(
                self._z(total, self.W), self._z(total), cols, latent, self._z(self.W, m.heads * dv),
                self._z(self.W, _up(l.ff, 16)) if l.ff else None))

    def _all_tensors(self) -> Iterator[torch.Tensor]:
        yield from (self.embed, self.head)
        if self.loop_in is not None:
            yield from (self.loop_in, self.loop_step)
        for w in self.weights:
            yield from (w.proj, w.bias, w.latent.norm, w.latent.ukv, w.o)
            if w.down is not None:
                yield w.down

    def weight_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self._all_tensors())

    # ------------------------------------------------------------------- loading
    def _place(self, name: str, t: torch.Tensor) -> bool:
        """Copy one checkpoint tensor into its padded place; False for a tensor the model has no use for."""
        width = self.arch.width

        def into(dst: torch.Tensor, src: torch.Tensor) -> None:
            dst.copy_(src.to(device=self.device, dtype=self.dtype))

        if name == "embed":
            into(self.embed[:, :width], t)
        elif name == "head":
            into(self.head[:, :width], t)
        elif name == "final.norm":
            self.final_gain = float(t)
        elif name == "loop.in":
            into(self.loop_in[:width, :width], t[:, :width])
            into(self.loop_in[:width, self.W:self.W + width], t[:, width:])
        elif name == "loop.step":
            into(self.loop_step[:, :width], t)
        else:
            index, _, sub = name[1:].partition(".")
            w, m = self.weights[int(index)], self.arch.layers[int(index)].mixer
            lw = w.latent

            def rows(section: str, n: int) -> torch.Tensor:
                lo = w.cols[section][0]
                return w.proj[lo:lo + n]

            def heads(mat: torch.Tensor, padded: int, real: int) -> torch.Tensor:
                return mat.view(m.heads, padded, mat.shape[1])[:, :real]

            if sub == "norm1":
                w.gain1 = float(t)
            elif sub == "norm2":
                w.gain2 = float(t)
            elif sub == "mix.q":
                into(heads(rows("q", m.heads * lw.dq), lw.dq, m.dim)[..., :width], t.view(m.heads, m.dim, width))
            elif sub == "mix.g":
                into(heads(rows("g", m.heads * lw.dv), lw.dv, m.vdim)[..., :width], t.view(m.heads, m.vdim, width))
            elif sub == "mix.dkv":
                into(rows("dkv", m.kv_rank)[:, :width], t)
            elif sub == "mix.dkv.norm":
                into(lw.norm, t)
            elif sub == "mix.uk":
                into(heads(lw.uk, lw.dq, m.dim)[..., :m.kv_rank], t.view(m.heads, m.dim, m.kv_rank))
            elif sub == "mix.uv":
                into(heads(lw.uv, lw.dv, m.vdim)[..., :m.kv_rank], t.view(m.heads, m.vdim, m.kv_rank))
            elif sub == "mix.o":
                into(w.o.view(self.W, m.heads, lw.dv)[:width, :, :m.vdim], t.view(width, m.heads, m.vdim))
            elif sub in ("rg1", "rg2"):
                into(rows(sub, width)[:, :width], t)
            elif sub in ("rg1.b", "rg2.b"):
                lo = w.cols[sub[:3]][0]
                into(w.bias[lo:lo + width], t)
            elif sub == "mlp.up":
                into(rows("up", t.shape[0])[:, :width], t)
            elif sub == "mlp.down":
                into(w.down[:width, :t.shape[1]], t)
            else:
                return False
        return True

    def load(self, tensors: Iterable[tuple[str, torch.Tensor]], *, strict: bool = True) -> None:
        """Copy checkpoint tensors into the packed, padded storage and bind the section tables."""
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
        self._bind()

    def _bind(self) -> None:
        for w in self.weights:
            gain = {"q": w.gain1, "dkv": w.gain1, "g": w.gain1, "rg1": w.gain1, "up": w.gain2, "rg2": w.gain2}
            act = {"q": None, "dkv": None, "g": "sigmoid", "rg1": "sigmoid", "up": "gelu", "rg2": "sigmoid"}
            w.sections = lat.Sections([(_up(n, 16), gain[s], act[s]) for s, (_, n) in w.cols.items()])
        cap = self.arch.logit_softcap
        self.head_sections = lat.Sections([(self.arch.vocab_size, self.final_gain, "softcap" if cap > 0 else None)], cap)

    # ---------------------------------------------------------------------- text
    @torch.no_grad()
    def forward(self, input_ids: torch.Tensor, positions: torch.Tensor, meta: AttnMeta, cache: "ops.KVCache", *,
                visual=None, vis_index=None, deepstack=None) -> torch.Tensor:
        """Rows ``[T, W]`` over their root mean square after the last layer run (the final gain is the head's)."""
        state = self.begin_layers(input_ids, positions, meta, cache, visual=visual, vis_index=vis_index, deepstack=deepstack)
        self.advance_layers(state, len(self.runs))
        return self.finish_layers(state)

    @torch.no_grad()
    def begin_layers(self, input_ids: torch.Tensor, positions: torch.Tensor, meta: AttnMeta, cache: "ops.KVCache", *,
                     visual=None, vis_index=None, deepstack=None) -> LayerLoopState:
        if visual is not None or deepstack:
            raise ValueError("the Poralorn family takes text only")
        T = input_ids.shape[0]
        x = torch.empty((T, self.W), dtype=torch.float32, device=self.device)
        n = torch.empty((T, self.W), dtype=self.dtype, device=self.device)
        pair = torch.empty((T, 2 * self.W), dtype=self.dtype, device=self.device) if self.loop_in is not None else None
        st = LayerLoopState(meta, cache, x, n, pair)
        lat.stream_update(x, self.arch.width, self.arch.norm_eps, keep=False, ids=input_ids, table=self.embed,
                          embed_out=pair[:, self.W:] if pair is not None else None, **self._outputs(st, 0))
        return st

    def _outputs(self, st: LayerLoopState, run: int) -> dict[str, torch.Tensor]:
        """What layer run ``run`` (or the head) reads: the stream itself where a pass begins, else its normalised rows."""
        if run < len(self.runs) and self.runs[run].loop_pass is not None:
            return {"raw_out": st.pair[:, :self.W]}
        return {"norm_out": st.n}

    @torch.no_grad()
    def advance_layers(self, st: LayerLoopState, max_layers: int) -> bool:
        """Run up to ``max_layers`` more layer runs; True once all have run."""
        a = self.arch
        stop = min(len(self.runs), st.next_layer + max(0, int(max_layers)))
        for i in range(st.next_layer, stop):
            run = self.runs[i]
            w = self.weights[run.layer]
            if run.loop_pass is not None:
                lat.stream_update(st.x, a.width, a.norm_eps, keep=False, a=lat.Branch(slabs=lat.linear_slabs(st.pair, self.loop_in)),
                                  bias=self.loop_step[run.loop_pass], norm_out=st.n)
            p = lat.linear_sections(st.n, w.proj, w.sections, bias=w.bias)
            ff = None
            if w.down is not None:
                ff = self._project(w.part(p, "up"), w.down)
                ff.gate = w.part(p, "rg2")
            mix = self._project(self._attend(p, w, st.meta, st.cache, i), w.o)
            mix.gate = w.part(p, "rg1")
            lat.stream_update(st.x, a.width, a.norm_eps, keep=True, a=mix, b=ff, mult=a.residual_mult, **self._outputs(st, i + 1))
        st.next_layer = stop
        return stop == len(self.runs)

    @torch.no_grad()
    def finish_layers(self, st: LayerLoopState) -> torch.Tensor:
        if st.next_layer != len(self.runs):
            raise RuntimeError(f"finish_layers after {st.next_layer} of {len(self.runs)} layer runs")
        return st.n

    def _project(self, x: torch.Tensor, w: torch.Tensor) -> lat.Branch:
        """Output projection of a sublayer: split-K slabs for up to a few hundred tokens, rows for long prompts."""
        if self.device.type == "cuda" and self.dtype == torch.float32:
            return lat.Branch(slabs=lat.linear_slabs(x, w))
        dense, partials, _ = self.comm.row_parallel(x, w)
        return lat.Branch(slabs=partials, rows=dense)

    def _attend(self, p: torch.Tensor, w: PoralornLayerWeights, meta: AttnMeta, cache: "ops.KVCache", slab: int) -> torch.Tensor:
        lw, eps = w.latent, self.arch.norm_eps
        q, raw, gate = (w.part(p, s) for s in ("q", "dkv", "g"))
        if not meta.is_prefill:
            return lat.latent_attention_absorbed(q, raw, gate, lw, eps, meta.slots, cache, slab, meta.block_tables, meta.context_lens)
        if p.is_cuda and p.dtype == torch.bfloat16 and lat.expanded_is_cheaper(lw, self.Rc, meta.total_kv, meta.attended_pairs):
            return lat.latent_attention_expanded(q, raw, gate, lw, eps, meta.slots, cache, slab, meta.block_tables, meta.cu_seqlens_q,
                                                 meta.max_q_len, cu_seqlens_kv=None if meta.no_history else meta.cu_seqlens_kv,
                                                 total_kv=meta.total_kv, max_kv_len=meta.max_kv_len)
        return lat.latent_attention_absorbed(q, raw, gate, lw, eps, meta.slots, cache, slab, meta.block_tables, meta.kv_lens,
                                             cu_seqlens_q=meta.cu_seqlens_q, max_q_len=meta.max_q_len)

    @torch.no_grad()
    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        """fp32 logits ``[B, vocab]``, capped."""
        return lat.linear_sections(hidden, self.head, self.head_sections, out_f32=True)

    @torch.no_grad()
    def sample(self, hidden: torch.Tensor, temperature: Optional[torch.Tensor], *, seed: int = 0,
               step: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        logits = self.sampled_logits = self.logits(hidden)
        if self.keep_logits:
            self.last_logits = logits.clone()
        return ops.sample(logits, temperature, seed=seed, step=step, out=out)
