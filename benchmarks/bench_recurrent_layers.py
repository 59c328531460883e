"""Prefill and decode throughput of the Bokorax family (time mixing with a matrix state, causal attention with sink and bounded
scores, windowed attention with tied values, scored routing) beside the closest family, Dolidra's head-gated windowed attention
with routed experts, at equal layer sizes (random weights), and every kernel of a layer against its roofline.

    python bench.py --workload recurrent-layers [--sizes 2048,4096] [--steps K] [--warmup W]
    python -m benchmarks.bench_recurrent_layers --kernels-only

Rows as in ``bench_latent_layers.py``; ``like`` names the row of the same size that a kernel is compared with.  The recurrence
has no like kernel; its roofline is the slower of its bytes and its 32-bit arithmetic outside the tensor cores.
"""

from __future__ import annotations

import argparse
import json
import sys

import torch

from benchmarks import bench_latent_layers as base

LAYERS, VOCAB, WINDOW, STATE_DIM, RANK = base.LAYERS, base.VOCAB, 1024, 64, 64
# width -> (query heads, key heads, head width, experts, chosen, expert feed-forward)
SIZES = {2048: (16, 4, 128, 32, 4, 768), 4096: (32, 8, 128, 32, 4, 1536), 8192: (64, 16, 128, 32, 4, 3072)}
FP32_RATE = 148 * 128 * 2 * 1.965e9    # fused multiply-adds outside the tensor cores at the highest clock


def arch(width: int, kind: str):
    """``kind``: ``recurrent``, ``causal``, ``windowed`` (layers of one mixer), ``kept`` (the closest family)."""
    from prism_infer_b200.models.architecture import (NO_WINDOW, BokoraxArch, BokoraxLayer, DolidraArch, DolidraLayer, MixtureArch, RotaryArch,
                                                      TimeMixArch, WindowAttentionArch)

    H, G, D, E, top, EF = SIZES[width]
    common = dict(heads=H, kv_heads=G, dim=D, vdim=D, scale=D ** -0.5, qk_norm=True)
    if kind == "kept":
        mixer = WindowAttentionArch(**common, rot=RotaryArch(1e6, D), window=WINDOW, keep_first=16, gate=True)
        return DolidraArch(vocab_size=VOCAB, width=width, layers=(DolidraLayer(mixer, moe=MixtureArch(E, top, EF, EF)),) * LAYERS, side_dim=16)
    moe = MixtureArch(E, top, EF, EF, scored=True, groups=4, groups_kept=2, scale=2.5, shared_gate=True)
    mixer = {"recurrent": TimeMixArch(width // STATE_DIM, STATE_DIM, RANK),
             "causal": WindowAttentionArch(**common, rot=RotaryArch(1e6, D, 4.0), window=NO_WINDOW, gate=True, head_norm=True, softcap=30.0, sink=True),
             "windowed": WindowAttentionArch(**common, rot=RotaryArch(1e6, D), window=WINDOW, tied_values=True)}[kind]
    return BokoraxArch(vocab_size=VOCAB, width=width, layers=(BokoraxLayer(mixer, moe),) * LAYERS)


def model_rows(widths, batches, prompts, context: int, steps: int, warmup: int) -> list[dict]:
    rows = []
    for width in widths:
        for family in ("recurrent", "causal", "windowed", "kept"):
            runner = base.make_runner(arch(width, family), batches, context)
            head = {"width": width, "family": family, "layers": LAYERS, "weight_bytes": base.layer_bytes(runner)}
            for tokens in prompts:
                ms = base.prefill_ms(runner, tokens, max(3, steps // 4), warmup)
                rows.append({**head, "phase": "prefill", "tokens": tokens, "ms": round(ms, 4), "tok_per_s": round(tokens / ms * 1e3)})
            for batch in batches:
                ms = base.decode_ms(runner, batch, context, steps, warmup)
                rows.append({**head, "phase": "decode", "batch": batch, "context": context, "ms": round(ms, 4),
                             "tok_per_s": round(batch / ms * 1e3)})
            runner.exit()
            del runner
            torch.cuda.empty_cache()
    return rows


class Kernels(base.Kernels):
    def __init__(self, width: int, steps: int, warmup: int) -> None:
        super().__init__(width, steps, warmup)
        self.H, self.G, self.D, self.E, self.top, self.EF = SIZES[width]

    def specs(self):
        """(family, what it is, spec, rows of the queries alone)"""
        from prism_infer_b200.models.architecture import NO_WINDOW
        from prism_infer_b200.ops import window

        common = dict(heads=self.H, kv_heads=self.G, maps=1, dim=self.D, vdim=self.D, rot_dims=self.D, scale=self.D ** -0.5, eps=1e-6)
        return [("bokorax", "causal, cap, sink", window.WindowSpec(**common, window=NO_WINDOW, keep_first=0, gate=True, head_norm=True, softcap=30.0)),
                ("bokorax", "window, tied values", window.WindowSpec(**common, window=WINDOW, keep_first=0, gate=False, tied=True)),
                ("dolidra", "causal", window.WindowSpec(**common, window=NO_WINDOW, keep_first=0, gate=True)),
                ("dolidra", "window, kept tokens", window.WindowSpec(**common, window=WINDOW, keep_first=16, gate=True))]

    # ---- recurrence ----------------------------------------------------------------------------------
    def recurrence(self, tokens: int, batch: int = 1) -> None:
        """``batch`` sequences of ``tokens`` each; one token: a decode step."""
        from prism_infer_b200.ops import latent as lat
        from prism_infer_b200.ops import native
        from prism_infer_b200.ops import recurrent as rec

        dev, W, n = "cuda", self.width, STATE_DIM
        H, T, decode = W // n, tokens * batch, tokens == 1
        sp = rec.TimeMixSpec(H, n, RANK, W, 1e-6)
        C = sp.cols
        tag = f"batch {batch}" if decode else f"{tokens} tokens" + (f" x {batch}" if batch > 1 else "")
        state_bytes = batch * (sp.carry + W) * 4
        sets = self.sets_for(2 * state_bytes if decode else 4 * C * W * 2)
        cache = rec.StateCache([sp.carry + W] * sets, batch, dev)
        x = torch.randn(T, W, device=dev)
        ws = [rec.TimeMixWeights(torch.rand(5, W, device=dev).bfloat16(), self.matrix(4 * C, W).view(4, C, W), self.matrix(RANK, W),
                                 self.matrix(C, RANK), torch.full((C,), -2.0, device=dev).bfloat16(), self.matrix(1, C)[0], self.matrix(1, C)[0])
              for _ in range(min(sets, 8))]
        slots = torch.arange(batch, dtype=torch.int32, device=dev)
        lens = torch.full((batch,), 64 + tokens, dtype=torch.int32, device=dev)
        cu = None if decode else (torch.arange(batch + 1, dtype=torch.int32, device=dev) * tokens)
        views = [rec.StateView(cache, i, slots, lens, cu) for i in range(sets)]
        w = lambda i: ws[i % len(ws)]  # noqa: E731
        st = lambda: torch.cuda.current_stream().cuda_stream  # noqa: E731
        mixed, table, keep = rec.token_mix(x, sp, w(0), views[0])
        out = torch.empty(T, C, device=dev, dtype=torch.bfloat16)
        self.time("bokorax", f"blends with the previous token, {tag}", "residual + norm", lambda i: rec.token_mix(x, sp, w(i), views[i]), sets,
                  T * W * (4 + 5 * 2))
        p = rec.wide_projections(mixed, w(0).rkvg, table)
        wide_out = p.slabs.numel() * 4 if p.slabs is not None else p.rows.numel() * 2
        self.time("bokorax", f"four projections, {tag}", "stacked projection", lambda i: rec.wide_projections(mixed, w(i).rkvg, table),
                  len(ws), 4 * C * W * 2 + 4 * T * W * 2 + wide_out, 8.0 * C * W * T)
        z1 = lat.linear_slabs(mixed[4], w(0).w1)
        self.time("bokorax", f"decay projection, narrow, {tag}", "router logits", lambda i: lat.linear_slabs(mixed[4], w(i).w1), len(ws),
                  RANK * W * 2 + T * (W * 2 + RANK * 4))
        z1_args, p_args = rec._proj_args(lat.Branch(slabs=z1)), rec._proj_args(p)
        if decode:
            def step(i):
                m = w(i)
                native.call("prism_state_step", 0, *views[i].args(sp, cu=False), x.data_ptr(), batch, W, *p_args, *z1_args, m.w2.data_ptr(),
                            m.w0.data_ptr(), m.u.data_ptr(), m.norm.data_ptr(), out.data_ptr(), H, n, n, RANK, 1e-6, st(), rec._pdl())

            self.time("bokorax", f"state step, {tag}", "", step, sets, 2 * state_bytes + wide_out + C * (RANK + 3) * 2 + batch * C * 2)
            return
        d = rec.decays(z1, w(0))
        self.time("bokorax", f"decays, {tag}", "stacked projection", lambda i: rec.decays(z1, w(i)), len(ws),
                  C * RANK * 2 + z1.numel() * 4 + T * C * 4, 4.0 * C * RANK * T)
        o = torch.empty(T, C, device=dev)

        def scan(i):
            native.call("prism_state_scan", 0, *views[i].args(sp), x.data_ptr(), batch, W, *p_args, d.data_ptr(), w(i).u.data_ptr(), o.data_ptr(), T, H,
                        n, st(), rec._pdl())

        # per state element: output product, decay product, key-value product and their sums
        self.time("bokorax", f"state scan, {tag}", "", scan, min(sets, 8), T * C * (3 * 2 + 4 + 4) + 2 * state_bytes, 5.0 * T * C * n, FP32_RATE)
        self.time("bokorax", f"norm per head and gate, {tag}", "residual + norm", lambda i: native.call(
            "prism_head_norm_gate", 0, o.data_ptr(), *p_args, w(i).norm.data_ptr(), out.data_ptr(), T, H, n, n, 1e-6, st(), rec._pdl()), 4, T * C * 8)

    # ---- stacked projection of an attention layer, router, residual ------------------------------------
    def shared(self, tokens: int) -> None:
        from prism_infer_b200.models.common import TPComm
        from prism_infer_b200.ops import latent as lat
        from prism_infer_b200.ops import moe

        W, E, K, comm, tag = self.width, self.E, self.top + 1, TPComm(), f"{tokens} tokens"
        small = tokens <= 128
        x = self.matrix(tokens, W)
        M = (self.H + 2 * self.G) * self.D + self.H
        n = self.sets_for(M * W * 2)
        ws = [self.matrix(M, W) for _ in range(n)]
        self.time("dolidra", f"stacked projection, {tag}", "", lambda i: comm.row_parallel(x, ws[i]), n,
                  M * W * 2 + tokens * (W * 2 + M * (4 if small else 2)), 2.0 * M * W * tokens)
        del ws
        slots = torch.arange(tokens, device="cuda")
        router = [self.matrix(E + 1, W) for _ in range(8)]
        self.time("dolidra", f"router logits, {tag}", "", lambda i: lat.linear_slabs(x, router[i][:E]), 8, E * W * 2 + tokens * (W * 2 + E * 4))
        self.time("bokorax", f"router logits, {tag}", "router logits", lambda i: lat.linear_slabs(x, router[i]), 8, E * W * 2 + tokens * (W * 2 + E * 4))
        logits = torch.randn(1, tokens, E + 1, device="cuda")
        own = moe.Scored(torch.zeros(E, device="cuda"), 8, 4, 2, 2.5, True)
        self.time("dolidra", f"routing, {tag}", "", lambda i: moe.route(lat.Branch(slabs=logits[..., :E]), self.top, E, 1, slots), 4, tokens * E * 4)
        self.time("bokorax", f"routing, {tag}", "routing", lambda i: moe.route(lat.Branch(slabs=logits), self.top, E - 8, 1, slots, scored=own), 4,
                  tokens * E * 4)
        w = torch.ones(W, device="cuda", dtype=torch.bfloat16)
        n = self.sets_for(tokens * W * 16)
        data = [dict(x=torch.zeros(tokens, W, device="cuda"), n=self.matrix(tokens, W)) for _ in range(n)]
        for family, r in (("dolidra", moe.route(lat.Branch(slabs=logits[..., :E]), self.top, E, 1, slots)),
                          ("bokorax", moe.route(lat.Branch(slabs=logits), self.top, E - 8, 1, slots, scored=own))):
            used = int((r.pos >= 0).sum())
            y = [torch.zeros(1, tokens * K, W, device="cuda") if small else self.matrix(tokens * K, W) for _ in range(min(n, 8))]

            def pairs(i, r=r, y=y, offset=1.0 if family == "bokorax" else 0.0):
                t = y[i % len(y)]
                b = lat.Branch(slabs=t if small else None, rows=None if small else t, pos=r.pos, weight=r.weight, post_norm=w, self_weight=r.self_weight)
                lat.stream_update(data[i]["x"], W, 1e-5, keep=True, a=b, raw_out=data[i]["n"], norm_offset=offset)

            self.time(family, f"expert sum + norm + residual, {tag}", "expert sum + norm + residual" if family == "bokorax" else "", pairs, n,
                      used * W * (4 if small else 2) + tokens * W * (8 + 2))
            del y

    # ---- attention -------------------------------------------------------------------------------------
    def decode_attention(self, batch: int, context: int) -> None:
        from prism_infer_b200 import ops
        from prism_infer_b200.ops import latent as lat
        from prism_infer_b200.ops import window

        page, dev = 256, "cuda"
        per_seq = -(-context // page)
        lens = torch.full((batch,), context, dtype=torch.int32, device=dev)
        table = torch.randperm(batch * per_seq, device=dev).to(torch.int32).view(batch, per_seq)
        slots = table[:, -1].long() * page + (context - 1) % page
        pos = torch.full((batch,), context - 1, dtype=torch.int32, device=dev)
        sink = torch.zeros(self.H, device=dev)
        for family, name, sp in self.specs():
            R = sp.k_cols + sp.v_cols
            keys = min(context, sp.window) + (min(sp.keep_first, max(0, context - sp.window)))
            n = self.sets_for(batch * keys * R * 2)
            cache = ops.KVCache(n, batch * per_seq, 1, page, R, ops.KV_BF16, dev, planes=1)
            for l in range(n):
                cache.token_rows(l).normal_()
            q = self.matrix(batch, sp.q_cols)
            gate = torch.rand(batch, sp.heads, device=dev) if sp.gate else None
            own = sink if sp.softcap else None
            self.time(family, f"decode attention ({name}), batch {batch}, {keys} keys", "decode attention" if family == "bokorax" else "",
                      lambda i: window.window_attention(q, sp, gate, cache, i, table, lens, sink=own), n, batch * keys * R * 2)
            if "causal" == name:
                continue
            self.prepare(family, name, sp, batch, torch.randn(2, batch, sp.proj_cols, device=dev), pos, slots, cache, n)
            del cache

    def prepare(self, family, name, sp, tokens, src, pos, slots, cache, n) -> None:
        from prism_infer_b200.ops import latent as lat
        from prism_infer_b200.ops import window

        slabs = src.dim() == 3
        one = lambda cols: torch.ones(self.D if sp.head_norm else cols, device="cuda", dtype=torch.bfloat16)  # noqa: E731
        w = window.WindowWeights(q_norm=one(sp.q_cols), k_norm=one(sp.k_cols), inv_freq=torch.rand(self.D // 2, device="cuda"))
        proj = lat.Branch(slabs=src) if slabs else lat.Branch(rows=src)
        self.time(family, f"prepare queries and cache rows ({name}), {tokens} tokens", "prepare" if family == "bokorax" else "",
                  lambda i: window.qkv_prepare(proj, sp, w, pos, slots, cache, i), n,
                  tokens * (sp.proj_cols * (8 if slabs else 2) + (sp.q_cols + sp.k_cols + sp.v_cols) * 2))

    def prefill_attention(self, tokens: int) -> None:
        from prism_infer_b200 import ops
        from prism_infer_b200.ops import window

        dev, D, page = "cuda", self.D, 256
        cu = torch.tensor([0, tokens], dtype=torch.int32, device=dev)
        lens = torch.tensor([tokens], dtype=torch.int32, device=dev)
        pages = -(-tokens // page)
        table = torch.arange(pages, dtype=torch.int32, device=dev).view(1, -1)
        slots, pos = torch.arange(tokens, device=dev), torch.arange(tokens, dtype=torch.int32, device=dev)
        sink = torch.zeros(self.H, device=dev)
        for family, name, sp in self.specs():
            w = min(sp.window, tokens)
            pairs = tokens * w - w * (w - 1) / 2
            R = sp.k_cols + sp.v_cols
            cache = ops.KVCache(2, pages, 1, page, R, ops.KV_BF16, dev, planes=1)
            for l in range(2):
                cache.token_rows(l).normal_()
            for spread in ((1.0, 20.0) if sp.softcap else (1.0,)):   # scores of about one, and scores that reach the bound
                q = torch.randn(tokens, sp.q_cols, device=dev, dtype=torch.bfloat16) * spread
                gate = torch.rand(tokens, sp.heads, device=dev) if sp.gate else None
                own = sink if sp.softcap else None
                tag = ", scores at the bound" if spread > 1 else ""
                self.time(family, f"prefill attention ({name}{tag}), {tokens} tokens", "prefill attention" if family == "bokorax" else "",
                          lambda i: window.window_attention(q, sp, gate, cache, i, table, lens, cu_seqlens_q=cu, max_q_len=tokens, sink=own), 2, 0,
                          4.0 * pairs * sp.heads * D)
            if "causal" == name:
                continue
            self.prepare(family, name, sp, tokens, self.matrix(tokens, sp.proj_cols), pos, slots, cache, 2)
            del cache
        q3, k3 = torch.randn(tokens, self.H, D, device=dev, dtype=torch.bfloat16), self.matrix(tokens, 2 * self.G * D).view(tokens, 2 * self.G, D)
        self.time("grouped", f"prefill attention (causal), {tokens} tokens", "",
                  lambda _: ops.varlen_attention(q3, k3[:, :self.G], k3[:, self.G:], cu, tokens, causal=True), 2, 0, 2.0 * tokens * tokens * self.H * D)


def kernel_rows(widths, steps: int, warmup: int) -> list[dict]:
    from prism_infer_b200 import ops
    from prism_infer_b200.ops import native

    native.lib()
    ops.set_pdl(True)
    ops.apply_tuning()
    rows = []
    for width in widths:
        k = Kernels(width, steps, warmup)
        for tokens, batch in ((1, 1), (1, 32), (1, 128), (2048, 1), (8192, 1), (2048, 4)):
            k.recurrence(tokens, batch)
            torch.cuda.empty_cache()
        for tokens in (1, 32, 2048):
            k.shared(tokens)
            torch.cuda.empty_cache()
        for batch, context in ((1, 2048), (32, 2048), (128, 2048)):
            k.decode_attention(batch, context)
            torch.cuda.empty_cache()
        for tokens in (2048, 8192):
            k.prefill_attention(tokens)
            torch.cuda.empty_cache()
        rows += k.rows
        del k
        torch.cuda.empty_cache()
    native.check_status()
    return rows


def main(argv: list[str] | None = None) -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--sizes", default="2048,4096")
    ap.add_argument("--batches", default="1,8,32,128")
    ap.add_argument("--prompts", default="512,2048,8192")
    ap.add_argument("--context", type=int, default=2048)
    ap.add_argument("--steps", type=int, default=40)
    ap.add_argument("--warmup", type=int, default=5)
    ap.add_argument("--kernels-only", action="store_true")
    ap.add_argument("--models-only", action="store_true")
    ap.add_argument("--output", default=None)
    args = ap.parse_args(argv)
    ints = lambda s: [int(v) for v in s.split(",")]  # noqa: E731
    widths = ints(args.sizes)
    from bench import ClockSampler

    sampler = ClockSampler(0)
    sampler.start()
    models = [] if args.kernels_only else model_rows(widths, ints(args.batches), ints(args.prompts), args.context, args.steps, max(3, args.warmup))
    kernels = [] if args.models_only else kernel_rows(widths, args.steps, max(3, args.warmup))
    out = {"workload": "recurrent-layers", "data": "synthetic (random weights and token ids)", "dtype": "bf16", "window": WINDOW,
           "l2": "operand sets or weights larger than L2", "models": models, "kernels": kernels, "clocks": sampler.stop()}
    text = json.dumps(out)
    if args.output:
        with open(args.output, "w", encoding="utf-8") as fh:
            fh.write(text + "\n")
    print(text)
    return 0


if __name__ == "__main__":
    sys.exit(main())
