"""Prefill and decode throughput of the Dolidra family (windowed differential attention, head-gated attention with kept first
tokens, mixture of experts) beside the grouped-query family at equal layer sizes (random weights), and every kernel of a layer
against its roofline.

    python bench.py --workload window-layers [--sizes 2048,4096] [--steps K] [--warmup W]
    python -m benchmarks.bench_window_layers --kernels-only

Rows as in ``bench_latent_layers.py``.  The grouped family has as many query and key heads of the same width; where the new
family sees a window, its like kernel gets a context of the window's length.
"""

from __future__ import annotations

import argparse
import json
import sys

import torch

from benchmarks import bench_latent_layers as base

LAYERS, VOCAB, WINDOW, KEEP, SIDE = base.LAYERS, base.VOCAB, 1024, 16, 256
# width -> (query heads of the one-map mixer, key heads, head width, feed-forward, experts, chosen, expert feed-forward)
SIZES = {2048: (16, 4, 128, 6144, 32, 4, 768), 4096: (32, 8, 128, 12288, 32, 4, 1536), 8192: (64, 16, 128, 24576, 32, 4, 3072)}


def arch(width: int, kind: str):
    """``kind``: ``maps`` / ``kept`` (dense layers of one mixer), ``experts`` (kept mixer, routed feed-forward)."""
    from prism_infer_b200.models.architecture import DolidraArch, DolidraLayer, MixtureArch, RotaryArch, WindowAttentionArch

    H, G, D, F, E, top, EF = SIZES[width]
    common = dict(dim=D, vdim=D, scale=D ** -0.5, rot=RotaryArch(1e6, D), window=WINDOW)
    mixer = (WindowAttentionArch(heads=H // 2, kv_heads=G // 2, maps=2, diff=0.5, bias=True, **common) if kind == "maps"
             else WindowAttentionArch(heads=H, kv_heads=G, keep_first=KEEP, qk_norm=True, gate=True, **common))
    layer = DolidraLayer(mixer, moe=MixtureArch(E, top, EF, EF)) if kind == "experts" else DolidraLayer(mixer, ff=F)
    return DolidraArch(vocab_size=VOCAB, width=width, layers=(layer,) * LAYERS, side_dim=SIDE)


def model_rows(widths, batches, prompts, context: int, steps: int, warmup: int) -> list[dict]:
    rows = []
    for width in widths:
        for family in ("maps", "kept", "experts", "grouped"):
            runner = base.make_runner(base.grouped_arch(width) if family == "grouped" else arch(width, family), batches, context)
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
        self.H, self.G, self.D, self.F, self.E, self.top, self.EF = SIZES[width]

    def spec(self, maps: int):
        from prism_infer_b200.ops import window

        H, G = (self.H // 2, self.G // 2) if maps == 2 else (self.H, self.G)
        return window.WindowSpec(heads=H, kv_heads=G, maps=maps, dim=self.D, vdim=self.D, rot_dims=self.D, scale=self.D ** -0.5, window=WINDOW,
                                 keep_first=0 if maps == 2 else KEEP, gate=maps == 1, eps=1e-5, lam=0.5, gain=0.5)

    # ---- feed-forwards -----------------------------------------------------------------------------
    def feed_forward(self, tokens: int) -> None:
        from prism_infer_b200 import ops
        from prism_infer_b200.models.common import TPComm
        from prism_infer_b200.ops import latent as lat
        from prism_infer_b200.ops import moe, native

        W, F, E, EF, K = self.width, self.F, self.E, self.EF, self.top + 1
        x, tag, comm = self.matrix(tokens, W), f"{tokens} tokens", TPComm()
        small = tokens <= 128
        n = self.sets_for(2 * F * W * 2)
        ws = [self.matrix(2 * F, W) for _ in range(n)]
        moved = 2 * F * W * 2 + tokens * (W + F) * 2
        self.time("dolidra", f"gate/up projection, tanh GELU, {tag}", "gate/up projection", lambda i: ops.gate_up_glu(x, ws[i], "gelu_tanh"), n,
                  moved, 4.0 * F * W * tokens)
        self.time("grouped", f"gate/up projection, {tag}", "", lambda i: ops.gate_up_swiglu(x, ws[i]), n, moved, 4.0 * F * W * tokens)
        f = self.matrix(tokens, F)
        self.time("grouped", f"down projection, {tag}", "", lambda i: comm.row_parallel(f, ws[i].view(W, -1)[:, :F]), n,
                  F * W * 2 + tokens * (F * 2 + W * (4 if small else 2)), 2.0 * F * W * tokens)
        del ws
        # routed: the experts that the tokens choose, at least one tile each
        logits = torch.randn(1, tokens, E, device="cuda")
        slots = torch.arange(tokens, device="cuda")
        r = moe.route(lat.Branch(slabs=logits), self.top, E, 1, slots)
        used = len({int(e) for e in r.groups[:int(r.n_groups[0]), 0].tolist()})
        n = self.sets_for(E * 2 * EF * W * 2)
        gu = [self.matrix((E + 1) * 2 * EF, W).view(E + 1, 2 * EF, W) for _ in range(n)]
        N = tokens * K
        a = self.matrix(N, EF)
        table = (r.groups.data_ptr(), r.groups.shape[0], r.n_groups.data_ptr())
        st = lambda: torch.cuda.current_stream().cuda_stream  # noqa: E731
        rows = self.matrix(N, W)
        y = torch.empty(4, N, W, device="cuda") if small else torch.empty(N, W, device="cuda", dtype=torch.bfloat16)
        splits = ops.effective_splits(EF, moe._down_splits(W, EF, r.groups.shape[0]))

        def up(i):
            if small:
                native.call("prism_gemm_grouped_small", gu[i].data_ptr(), x.data_ptr(), a.data_ptr(), EF, tokens, tokens, W, W, EF, *table,
                            r.row_token.data_ptr(), N, E + 1, 1, 1, 0, st(), ops._pdl())
            else:
                native.call("prism_gemm_grouped", gu[i].data_ptr(), rows.data_ptr(), a.data_ptr(), EF, N, W, W, EF, *table, E + 1, 1, st(),
                            ops._pdl())

        def down(i):
            w = gu[i].data_ptr()
            if small:
                native.call("prism_gemm_grouped_small", w, a.data_ptr(), y.data_ptr(), W, tokens, N, EF, EF, W, *table, None, N, E + 1, 0, splits,
                            N * W, st(), ops._pdl())
            else:
                native.call("prism_gemm_grouped", w, a.data_ptr(), y.data_ptr(), W, N, EF, EF, W, *table, E + 1, 0, st(), ops._pdl())

        self.time("dolidra", f"experts gate/up, {tag}", "gate/up projection", up, n,
                  used * 2 * EF * W * 2 + (tokens if small else N) * W * 2 + N * EF * 2, 4.0 * EF * W * N)
        self.time("dolidra", f"experts down, {tag}", "down projection", down, n,
                  used * EF * W * 2 + N * (EF * 2 + W * (4 * splits if small else 2)), 2.0 * EF * W * N)
        self.time("dolidra", f"routing, {tag}", "", lambda i: moe.route(lat.Branch(slabs=logits), self.top, E, 1, slots), 4, tokens * E * 4)
        if not small:
            self.time("dolidra", f"gather of expert rows, {tag}", "residual + norm", lambda i: native.call(
                "prism_moe_gather", x.data_ptr(), W, r.pos.data_ptr(), rows.data_ptr(), tokens, K, W, st(), ops._pdl()), 4, (tokens + N) * W * 2)
        del gu
        router = [self.matrix(E, W) for _ in range(8)]
        self.time("dolidra", f"router logits, {tag}", "", lambda i: lat.linear_slabs(x, router[i]), 8, E * W * 2 + tokens * (W * 2 + E * 4))
        n = self.sets_for(SIDE * W * 4)
        sw = [self.matrix(SIDE, W) for _ in range(n)]
        g = self.matrix(tokens, SIDE)
        self.time("dolidra", f"side gate projection, {tag}", "", lambda i: lat.linear_slabs(x, sw[i]), n, SIDE * W * 2 + tokens * (W * 2 + SIDE * 4))
        self.time("dolidra", f"side output projection, {tag}", "", lambda i: comm.row_parallel(g, sw[i].view(W, SIDE)), n,
                  SIDE * W * 2 + tokens * (W * (4 if small else 2) + SIDE * 2))

    # ---- residual ------------------------------------------------------------------------------------
    def residual(self, tokens: int) -> None:
        from prism_infer_b200 import ops
        from prism_infer_b200.ops import latent as lat
        from prism_infer_b200.ops import moe

        W, K = self.width, self.top + 1
        small = tokens <= 128
        P = ops.choose_splits(W, self.F, tokens) if small else 1
        w = torch.ones(W, device="cuda", dtype=torch.bfloat16)
        n = self.sets_for(tokens * W * (P * 4 + 16))
        data = [dict(x=torch.zeros(tokens, W, device="cuda"), n=self.matrix(tokens, W), r=self.matrix(tokens, W),
                     a=torch.zeros(P, tokens, W, device="cuda") if small else self.matrix(tokens, W)) for _ in range(n)]

        def branch(t):
            return lat.Branch(slabs=t, post_norm=w) if small else lat.Branch(rows=t, post_norm=w)

        def stream(i):
            d = data[i]
            lat.stream_update(d["x"], W, 1e-5, keep=True, a=branch(d["a"]), norm_weight=w, norm_out=d["n"])

        moved = tokens * W * ((P * 4 if small else 2) + 8 + 2)
        self.time("dolidra", f"norm + residual + norm, {tokens} tokens", "residual + norm", stream, n, moved)

        def addnorm(i):
            d = data[i]
            ops.add_rmsnorm(w, 1e-6, x=None if small else d["a"], partials=d["a"] if small else None, residual=d["r"])

        self.time("grouped", f"residual + norm, {tokens} tokens", "", addnorm, n, tokens * W * ((P * 4 if small else 2) + 6))
        r = moe.route(lat.Branch(slabs=torch.randn(1, tokens, self.E, device="cuda")), self.top, self.E, 1, torch.arange(tokens, device="cuda"))
        y = [torch.zeros(1, tokens * K, W, device="cuda") if small else self.matrix(tokens * K, W) for _ in range(min(n, 8))]

        def pairs(i):
            t = y[i % len(y)]
            b = lat.Branch(slabs=t if small else None, rows=None if small else t, pos=r.pos, weight=r.weight, post_norm=w)
            lat.stream_update(data[i]["x"], W, 1e-5, keep=True, a=b, raw_out=data[i]["n"])

        self.time("dolidra", f"expert sum + norm + residual, {tokens} tokens", "residual + norm", pairs, n,
                  tokens * W * (K * (4 if small else 2) + 8 + 2))

    # ---- attention -------------------------------------------------------------------------------------
    def decode_attention(self, batch: int, context: int) -> None:
        from prism_infer_b200 import ops
        from prism_infer_b200.ops import latent as lat
        from prism_infer_b200.ops import window

        page, dev, D = 256, "cuda", self.D
        per_seq = -(-context // page)
        lens = torch.full((batch,), context, dtype=torch.int32, device=dev)
        table = torch.randperm(batch * per_seq, device=dev).to(torch.int32).view(batch, per_seq)
        slots = table[:, -1].long() * page + (context - 1) % page
        pos = torch.full((batch,), context - 1, dtype=torch.int32, device=dev)
        seen = min(context, WINDOW)
        for maps in (1, 2):
            sp = self.spec(maps)
            R = sp.k_cols + sp.v_cols
            keys = seen + (min(KEEP, context - seen) if maps == 1 else 0)
            nbytes = batch * keys * R * 2
            n = self.sets_for(nbytes)
            cache = ops.KVCache(n, batch * per_seq, 1, page, R, ops.KV_BF16, dev, planes=1)
            for l in range(n):
                cache.token_rows(l).normal_()
            q = self.matrix(batch, sp.q_cols)
            gate = torch.rand(batch, sp.heads, device=dev) if sp.gate else None
            name = "two maps" if maps == 2 else "kept tokens, gate"
            self.time("dolidra", f"windowed decode attention ({name}), batch {batch}, {context} keys", "paged decode attention",
                      lambda i: window.window_attention(q, sp, gate, cache, i, table, lens), n, nbytes)
            proj = torch.randn(2, batch, sp.proj_cols, device=dev)
            w = window.WindowWeights(bias=torch.zeros(sp.proj_cols, device=dev, dtype=torch.bfloat16) if maps == 2 else None,
                                     q_norm=torch.ones(sp.q_cols, device=dev, dtype=torch.bfloat16) if maps == 1 else None,
                                     k_norm=torch.ones(sp.k_cols, device=dev, dtype=torch.bfloat16) if maps == 1 else None,
                                     inv_freq=torch.rand(D // 2, device=dev))
            self.time("dolidra", f"prepare queries and cache rows ({name}), batch {batch}", "QK norm + rotary + store",
                      lambda i: window.qkv_prepare(lat.Branch(slabs=proj), sp, w, pos, slots, cache, i), n,
                      batch * (sp.proj_cols * 8 + (sp.q_cols + R) * 2))
            del cache
        H, G = self.H, self.G
        g_bytes = batch * seen * G * D * 4
        n = self.sets_for(g_bytes)
        gc = ops.KVCache(n, batch * per_seq, G, page, D, ops.KV_BF16, dev)
        gc.payload.normal_()
        q3 = torch.randn(batch, H, D, device=dev, dtype=torch.bfloat16)
        partials = torch.randn(2, batch, (H + 2 * G) * D, device=dev)
        one = torch.ones(D, device=dev, dtype=torch.bfloat16)
        p3 = pos.repeat(3, 1).contiguous()
        short = torch.full((batch,), seen, dtype=torch.int32, device=dev)
        self.time("grouped", f"paged decode attention, batch {batch}, {seen} keys", "",
                  lambda i: ops.paged_decode_attention(q3, gc, i, table, short), n, g_bytes)
        self.time("grouped", f"QK norm + rotary + store, batch {batch}", "", lambda i: ops.qk_norm_rope_store(
            qkv=None, partials=partials, positions=p3, q_weight=one, k_weight=one, num_heads=H, num_kv_heads=G, head_dim=D, theta=1e6,
            section=(24, 20, 20), eps=1e-6, slots=slots, cache=gc, layer=i), n, batch * (H + 2 * G) * D * 12)

    def prefill_attention(self, tokens: int) -> None:
        from prism_infer_b200 import ops
        from prism_infer_b200.ops import latent as lat
        from prism_infer_b200.ops import window

        dev, D, page = "cuda", self.D, 256
        cu = torch.tensor([0, tokens], dtype=torch.int32, device=dev)
        lens = torch.tensor([tokens], dtype=torch.int32, device=dev)
        pages = -(-tokens // page)
        table = torch.arange(pages, dtype=torch.int32, device=dev).view(1, -1)
        slots, pos = torch.arange(tokens, device=dev), torch.arange(tokens, dtype=torch.int32, device=dev)
        pairs = tokens * (tokens + 1) / 2 if tokens <= WINDOW else tokens * WINDOW - WINDOW * (WINDOW - 1) / 2
        for maps in (1, 2):
            sp = self.spec(maps)
            R = sp.k_cols + sp.v_cols
            cache = ops.KVCache(2, pages, 1, page, R, ops.KV_BF16, dev, planes=1)
            for l in range(2):
                cache.token_rows(l).normal_()
            q = self.matrix(tokens, sp.q_cols) * 10
            gate = torch.rand(tokens, sp.heads, device=dev) if sp.gate else None
            name = "two maps" if maps == 2 else "kept tokens, gate"
            self.time("dolidra", f"windowed attention ({name}), {tokens} tokens", "causal attention",
                      lambda i: window.window_attention(q, sp, gate, cache, i, table, lens, cu_seqlens_q=cu, max_q_len=tokens), 2, 0,
                      4.0 * pairs * sp.heads * maps * D)
            proj = self.matrix(tokens, sp.proj_cols)
            w = window.WindowWeights(bias=torch.zeros(sp.proj_cols, device=dev, dtype=torch.bfloat16) if maps == 2 else None,
                                     q_norm=torch.ones(sp.q_cols, device=dev, dtype=torch.bfloat16) if maps == 1 else None,
                                     k_norm=torch.ones(sp.k_cols, device=dev, dtype=torch.bfloat16) if maps == 1 else None,
                                     inv_freq=torch.rand(D // 2, device=dev))
            self.time("dolidra", f"prepare queries and cache rows ({name}), {tokens} tokens", "QK norm + rotary + store",
                      lambda i: window.qkv_prepare(lat.Branch(rows=proj), sp, w, pos, slots, cache, i), 2,
                      tokens * (sp.proj_cols * 2 + (sp.q_cols + R) * 2))
            del cache
        H, G = self.H, self.G
        q3, k3 = (self.matrix(tokens, H * D) * 10).view(tokens, H, D), self.matrix(tokens, 2 * G * D).view(tokens, 2 * G, D)
        self.time("grouped", f"causal attention, {tokens} tokens", "", lambda _: ops.varlen_attention(q3, k3[:, :G], k3[:, G:], cu, tokens, causal=True),
                  2, 0, 2.0 * tokens * tokens * H * D)
        gc = ops.KVCache(2, pages, G, page, D, ops.KV_BF16, dev)
        qkv, one = self.matrix(tokens, (H + 2 * G) * D), torch.ones(D, device=dev, dtype=torch.bfloat16)
        p3 = pos.repeat(3, 1).contiguous()
        self.time("grouped", f"QK norm + rotary + store, {tokens} tokens", "", lambda i: ops.qk_norm_rope_store(
            qkv=qkv, partials=None, positions=p3, q_weight=one, k_weight=one, num_heads=H, num_kv_heads=G, head_dim=D, theta=1e6,
            section=(24, 20, 20), eps=1e-6, slots=slots, cache=gc, layer=i), 2, tokens * (2 * H + 4 * G) * D * 2)


def kernel_rows(widths, steps: int, warmup: int) -> list[dict]:
    from prism_infer_b200 import ops
    from prism_infer_b200.ops import native

    native.lib()
    ops.set_pdl(True)
    ops.apply_tuning()
    rows = []
    for width in widths:
        k = Kernels(width, steps, warmup)
        for tokens in (1, 32, 2048):
            k.feed_forward(tokens)
            k.residual(tokens)
            torch.cuda.empty_cache()
        for batch, context in ((1, 2048), (32, 2048), (128, 2048)):
            k.decode_attention(batch, context)
            torch.cuda.empty_cache()
        for tokens in (2048, 8192):
            k.prefill_attention(tokens)
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
    out = {"workload": "window-layers", "data": "synthetic (random weights and token ids)", "dtype": "bf16", "window": WINDOW,
           "l2": "operand sets or weights larger than L2", "models": models, "kernels": kernels, "clocks": sampler.stop()}
    text = json.dumps(out)
    if args.output:
        with open(args.output, "w", encoding="utf-8") as fh:
            fh.write(text + "\n")
    print(text)
    return 0


if __name__ == "__main__":
    sys.exit(main())
