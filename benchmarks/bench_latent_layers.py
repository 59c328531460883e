"""Prefill and decode throughput of the latent-attention family beside the grouped-query family at equal layer sizes
(random weights), and every kernel of a layer against its roofline.

    python bench.py --workload latent-layers [--sizes 2048,4096] [--steps K] [--warmup W]
    python -m benchmarks.bench_latent_layers --kernels-only

Model rows: four layers of each family through the engine's own model runner - prefill of one prompt timed with CUDA
events around whole forwards, decode as back-to-back launches of the captured graph (four layers of weights are
larger than L2).  Kernel rows: CUDA events around one op over rotating operand sets larger than L2; achieved bytes or
FLOPs over the measured copy bandwidth or bf16 GEMM rate of ``MEASURED_PEAKS.json``.
"""

from __future__ import annotations

import argparse
import json
import os
import sys

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
if ROOT not in sys.path:
    sys.path.insert(0, ROOT)

LAYERS = 4
VOCAB = 32_768
# width -> (heads, head width, latent width, feed-forward width)
SIZES = {2048: (16, 128, 256, 6144), 4096: (32, 128, 512, 12288), 8192: (64, 128, 512, 24576)}
L2_BYTES = 126 << 20


def peaks() -> tuple[float, float]:
    """(copy bandwidth in bytes/s, bf16 rate in FLOP/s)"""
    try:
        with open(os.path.join(ROOT, "MEASURED_PEAKS.json"), encoding="utf-8") as fh:
            p = json.load(fh)
        return p["hbm_gbs"] * 1e9, p["bf16_tflops"] * 1e12
    except (OSError, KeyError):
        return 6.65e12, 1.59e15


def latent_arch(width: int):
    from prism_infer_b200.models.architecture import PoralornArch

    heads, dim, rank, ff = SIZES[width]
    return PoralornArch.like_8b(LAYERS, width=width, heads=heads, dim=dim, kv_rank=rank, ff=ff, vocab_size=VOCAB)


def grouped_arch(width: int):
    from prism_infer_b200.models.architecture import Qwen3VLArch, TextArch, VisionArch

    heads, dim, _, ff = SIZES[width]
    return Qwen3VLArch(
        text=TextArch(vocab_size=VOCAB, hidden_size=width, num_layers=LAYERS, num_heads=heads, num_kv_heads=heads // 4, head_dim=dim,
                      intermediate_size=ff),
        vision=VisionArch(hidden_size=128, depth=1, num_heads=4, intermediate_size=256, num_position_embeddings=256,
                          out_hidden_size=width, deepstack_visual_indexes=(0,)),
        image_token_id=VOCAB - 1, video_token_id=VOCAB - 2, vision_start_token_id=VOCAB - 3, vision_end_token_id=VOCAB - 4,
        eos_token_id=VOCAB - 5)


def make_runner(arch, batches, context: int, page: int = 256):
    from prism_infer_b200.config import Config
    from prism_infer_b200.engine.model_runner import ModelRunner

    per_seq = -(-(context + 8) // page)
    cfg = Config("random:bench", arch=arch, max_model_len=per_seq * page, kvcache_block_size=page,
                 num_kvcache_blocks=per_seq * max(batches) + 1, cpu_kv_cache_ratio=0.0, max_num_seqs=max(batches), enable_decode_run_ahead=False)
    return ModelRunner(cfg, device="cuda:0")


def events_ms(fn, steps: int, warmup: int) -> float:
    for i in range(warmup):
        fn(i)
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for i in range(steps):
        fn(i)
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / steps


def prefill_ms(runner, tokens: int, steps: int, warmup: int) -> float:
    from prism_infer_b200.models.common import AttnMeta

    dev = runner.device
    pages = -(-tokens // runner.page)
    cache = runner._new_cache(pages, dev)
    ids = torch.randint(0, VOCAB - 8, (tokens,), device=dev)
    pos = torch.arange(tokens, dtype=torch.int32, device=dev).repeat(3, 1).contiguous()
    meta = AttnMeta(is_prefill=True, block_tables=torch.arange(pages, dtype=torch.int32, device=dev).view(1, -1),
                    slots=torch.arange(tokens, device=dev), cu_seqlens_q=torch.tensor([0, tokens], dtype=torch.int32, device=dev),
                    kv_lens=torch.tensor([tokens], dtype=torch.int32, device=dev), max_q_len=tokens, no_history=True, total_kv=tokens,
                    max_kv_len=tokens, attended_pairs=tokens * tokens, **runner._state_meta([0]))
    return events_ms(lambda _: runner.model.forward(ids, pos, meta, cache), steps, warmup)


def decode_ms(runner, batch: int, context: int, steps: int, warmup: int) -> float:
    from prism_infer_b200.engine.input_preparation import StepInputs

    per_seq = runner.max_blocks
    table = torch.arange(batch * per_seq, dtype=torch.int32).view(batch, per_seq)
    last = context - 1
    slots = table[:, last // runner.page].long() * runner.page + last % runner.page
    inp = StepInputs(kind="decode", input_ids=torch.randint(0, VOCAB - 8, (batch,)), positions=torch.full((3, batch), last, dtype=torch.int32),
                     slots=slots, block_tables=table, temperatures=torch.zeros(batch), context_lens=torch.full((batch,), context, dtype=torch.int32),
                     state_slots=torch.arange(batch, dtype=torch.int32) if runner.state is not None else None)
    runner.execute(inp)
    runner.time_decode_graph(warmup)
    return runner.time_decode_graph(steps)


def layer_bytes(runner) -> int:
    return runner.model.weight_bytes()


def model_rows(widths, batches, prompts, context: int, steps: int, warmup: int) -> list[dict]:
    rows = []
    for width in widths:
        for family, make in (("latent", latent_arch), ("grouped", grouped_arch)):
            runner = make_runner(make(width), batches, context)
            base = {"width": width, "family": family, "layers": LAYERS, "weight_bytes": layer_bytes(runner)}
            for tokens in prompts:
                ms = prefill_ms(runner, tokens, max(3, steps // 4), warmup)
                rows.append({**base, "phase": "prefill", "tokens": tokens, "ms": round(ms, 4), "tok_per_s": round(tokens / ms * 1e3)})
            for batch in batches:
                ms = decode_ms(runner, batch, context, steps, warmup)
                rows.append({**base, "phase": "decode", "batch": batch, "context": context, "ms": round(ms, 4),
                             "tok_per_s": round(batch / ms * 1e3)})
            runner.exit()
            del runner
            torch.cuda.empty_cache()
    return rows


# ------------------------------------------------------------------------------------------------ kernels
class Kernels:
    """Each op of a layer on its own.  ``nbytes``: bytes that must move, ``flops``: tensor work; the roofline is the
    slower of the two."""

    def __init__(self, width: int, steps: int, warmup: int) -> None:
        self.width, self.steps, self.warmup = width, steps, warmup
        self.heads, self.dim, self.rank, self.ff = SIZES[width]
        self.bw, self.rate = peaks()
        self.rows: list[dict] = []

    def time(self, family: str, name: str, like: str, fn, sets: int, nbytes: float, flops: float = 0.0, rate: float = 0.0) -> None:
        """``fn(i)`` runs operand set ``i``; ``sets`` of them together exceed L2.  ``rate``: FLOP/s of work that is not the tensor
        cores'."""
        graph_ms = self._graph(fn, sets)
        roof = max(nbytes / self.bw, flops / (rate or self.rate)) * 1e3
        self.rows.append({"width": self.width, "family": family, "kernel": name, "like": like, "us": round(graph_ms * 1e3, 2),
                          "roofline_us": round(roof * 1e3, 2), "fraction": round(roof / graph_ms, 3)})

    def _graph(self, fn, sets: int) -> float:
        """One pass over all sets as a captured graph (no host time between launches), replayed."""
        stream = torch.cuda.Stream()
        stream.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(stream):
            for i in range(sets):
                fn(i)
            stream.synchronize()
            g = torch.cuda.CUDAGraph()
            with torch.cuda.graph(g, stream=stream):
                for i in range(sets):
                    fn(i)
        torch.cuda.current_stream().wait_stream(stream)
        reps = max(3, self.steps // max(1, sets // 4))
        ms = events_ms(lambda _: g.replay(), reps, self.warmup) / sets
        del g
        return ms

    @staticmethod
    def sets_for(nbytes: float) -> int:
        return int(min(64, max(2, -(-2 * L2_BYTES // max(1, int(nbytes))))))

    def matrix(self, rows: int, cols: int) -> torch.Tensor:
        return (torch.randn(rows, cols, device="cuda", dtype=torch.bfloat16) * cols ** -0.5)

    # ---- projections -------------------------------------------------------------------------------
    def projections(self, tokens: int) -> None:
        from prism_infer_b200 import ops
        from prism_infer_b200.ops import latent as lat

        W, H, D, R, F = self.width, self.heads, self.dim, self.rank, self.ff
        x = self.matrix(tokens, W)
        parts = [(H * D, 0.9, None), (R, 0.9, None), (H * D, 0.9, "sigmoid"), (W, 0.9, "sigmoid"), (F, 1.1, "gelu"), (W, 1.1, "sigmoid")]
        M = sum(p[0] for p in parts)
        sec, bias = lat.Sections(parts), torch.zeros(M, device="cuda", dtype=torch.bfloat16)
        tag = f"{tokens} tokens"
        small = tokens <= 128

        def gemm(family, name, like, m, k, fn, out_bytes):
            n = self.sets_for(m * k * 2)
            ws = [self.matrix(m, k) for _ in range(n)]
            self.time(family, f"{name}, {tag}", like, lambda i: fn(ws[i]), n, m * k * 2 + tokens * k * 2 + out_bytes, 2.0 * m * k * tokens)

        gemm("latent", "stacked projection", "gate/up projection", M, W, lambda w: lat.linear_sections(x, w, sec, bias=bias), tokens * M * 2)
        gemm("grouped", "gate/up projection", "", 2 * F, W, lambda w: ops.gate_up_swiglu(x, w), tokens * F * 2)
        a, f = self.matrix(tokens, H * D), self.matrix(tokens, F)
        from prism_infer_b200.models.common import TPComm

        comm = TPComm()
        for family in ("latent", "grouped"):  # the same kernel in both families
            gemm(family, "attention output projection", "attention output projection", W, H * D, lambda w: comm.row_parallel(a, w),
                 tokens * W * (4 if small else 2))
            gemm(family, "down projection", "down projection", W, F, lambda w: comm.row_parallel(f, w), tokens * W * (4 if small else 2))
        both = self.matrix(tokens, 2 * W)
        gemm("latent", "loop projection", "attention output projection", W, 2 * W, lambda w: lat.linear_slabs(both, w), tokens * W * 4)
        if small:
            head = lat.Sections([(VOCAB, 1.0, "softcap")], 30.0)
            gemm("latent", "capped head", "head", VOCAB, W, lambda w: lat.linear_sections(x, w, head, out_f32=True), tokens * VOCAB * 4)
            gemm("grouped", "head", "", VOCAB, W, lambda w: ops.linear_partial(x, w, 1), tokens * VOCAB * 4)

    # ---- residual ------------------------------------------------------------------------------------
    def residual(self, tokens: int) -> None:
        from prism_infer_b200 import ops
        from prism_infer_b200.ops import latent as lat

        W = self.width
        small = tokens <= 128
        P = ops.choose_splits(W, self.ff, tokens) if small else 1
        P2 = ops.choose_splits(W, self.heads * self.dim, tokens) if small else 1
        per = tokens * W * ((P + P2) * 4 + 16 if small else 18)
        n = self.sets_for(per)
        data = []
        for _ in range(n):
            d = dict(x=torch.zeros(tokens, W, device="cuda"), n=self.matrix(tokens, W), g=self.matrix(tokens, 2 * W))
            if small:
                d.update(a=torch.zeros(P2, tokens, W, device="cuda"), b=torch.zeros(P, tokens, W, device="cuda"))
            else:
                d.update(a=self.matrix(tokens, W), b=self.matrix(tokens, W))
            data.append(d)

        def branch(d, k, lo):
            g = d["g"][:, lo:lo + W]
            return lat.Branch(slabs=d[k], gate=g) if small else lat.Branch(rows=d[k], gate=g)

        def stream(i):
            d = data[i]
            lat.stream_update(d["x"], W, 1e-5, keep=True, a=branch(d, "a", 0), b=branch(d, "b", W), mult=0.3, norm_out=d["n"])

        moved = tokens * W * ((P + P2) * 4 + 4 + 8 + 2) if small else tokens * W * (4 + 4 + 8 + 2)
        self.time("latent", f"gated residual + norm, {tokens} tokens", "residual + norm", stream, n, moved)
        w = torch.ones(W, device="cuda", dtype=torch.bfloat16)
        res = [self.matrix(tokens, W) for _ in range(n)]

        def addnorm(i):
            d = data[i]
            ops.add_rmsnorm(w, 1e-6, x=None if small else d["a"], partials=d["b"] if small else None, residual=res[i])

        self.time("grouped", f"residual + norm, {tokens} tokens", "", addnorm, n, tokens * W * ((P * 4 if small else 2) + 6))

    # ---- attention -------------------------------------------------------------------------------------
    def decode_attention(self, batch: int, context: int) -> None:
        from prism_infer_b200 import ops
        from prism_infer_b200.ops import latent as lat
        from prism_infer_b200.ops import native

        H, D, R = self.heads, self.dim, self.rank
        page, dev = 256, "cuda"
        per_seq = -(-context // page)
        lens = torch.full((batch,), context, dtype=torch.int32, device=dev)
        table = torch.randperm(batch * per_seq, device=dev).to(torch.int32).view(batch, per_seq)
        slots = table[:, -1].long() * page + (context - 1) % page
        tag = f"batch {batch}, {context} keys"
        kv_bytes = batch * context * R * 2
        n = self.sets_for(kv_bytes)
        cache = ops.KVCache(n, batch * per_seq, 1, page, R, ops.KV_BF16, dev, planes=1)
        cache.payload.normal_()
        ukv = [self.matrix(2 * H * D, R) for _ in range(n)]
        lws = [lat.LatentWeights(H, D, D, R, D ** -0.5, torch.ones(R, device=dev, dtype=torch.bfloat16), u) for u in ukv]
        q, raw, gate = self.matrix(batch, H * D), self.matrix(batch, R), self.matrix(batch, H * D)
        ns = lat.latent_splits(batch, H)
        qa = torch.randn(batch, H, R, device=dev, dtype=torch.bfloat16)
        po = torch.empty(batch * H, ns, R, device=dev) if ns > 1 else None
        ml = torch.zeros(batch * H, ns, 2, device=dev) if ns > 1 else None
        la = torch.empty(batch * H, R, device=dev, dtype=torch.bfloat16)
        out = torch.empty(batch, H * D, device=dev, dtype=torch.bfloat16)
        p, s, pdl = (lambda t: None if t is None else t.data_ptr()), (lambda: torch.cuda.current_stream().cuda_stream), ops._pdl

        def absorb(i):
            native.call("prism_latent_absorb", p(q), None, 0, 0, q.stride(0), *lat.NO_ROTARY, 0, 0, p(lws[i].uk), p(qa), p(raw), raw.stride(0), p(lws[i].norm), p(cache.latent(i)),
                        p(slots), cache.num_blocks * page, batch, H, D, R, R, 1e-5, s(), pdl())

        def attend(i):
            native.call("prism_latent_attention", p(qa), p(cache.latent(i)), p(table), None, p(lens), p(po), p(ml), p(la), batch, 1, H, R, R, page,
                        per_seq, cache.num_blocks, ns, lat.NO_WINDOW, D ** -0.5, s(), pdl())

        def output(i):
            native.call("prism_latent_out", p(po), p(ml), p(la), p(lws[i].uv), R, p(gate), gate.stride(0), p(out), out.stride(0), batch, H, D, R, ns,
                        s(), pdl())

        def whole(i):
            lat.latent_attention_absorbed(q, raw, gate, lws[i], 1e-5, slots, cache, i, table, lens)

        u_bytes = H * D * R * 2
        self.time("latent", f"absorb + latent store, {tag}", "QK norm + rotary + store", absorb, n, u_bytes + batch * H * (D + R) * 2)
        self.time("latent", f"latent attention, {tag}", "paged decode attention", attend, n, kv_bytes + batch * H * R * 4,
                  4.0 * batch * H * context * R)
        self.time("latent", f"merge + value up + gate, {tag}", "QK norm + rotary + store", output, n, u_bytes + batch * H * (R + D) * 2)
        self.time("latent", f"all three, {tag}", "store + decode attention", whole, n, 2 * u_bytes + kv_bytes, 4.0 * batch * H * context * R)
        del cache, ukv, lws
        Hkv = H // 4
        g_bytes = batch * context * Hkv * D * 4
        n = self.sets_for(g_bytes)
        gc = ops.KVCache(n, batch * per_seq, Hkv, page, D, ops.KV_BF16, dev)
        gc.payload.normal_()
        q3 = torch.randn(batch, H, D, device=dev, dtype=torch.bfloat16)
        qkv = self.matrix(batch, (H + 2 * Hkv) * D)
        one = torch.ones(D, device=dev, dtype=torch.bfloat16)
        pos = torch.zeros((3, batch), dtype=torch.int32, device=dev)

        def store(i):
            ops.qk_norm_rope_store(qkv=qkv, partials=None, positions=pos, q_weight=one, k_weight=one, num_heads=H, num_kv_heads=Hkv, head_dim=D,
                                   theta=1e6, section=(24, 20, 20), eps=1e-6, slots=slots, cache=gc, layer=i)

        def paged(i):
            ops.paged_decode_attention(q3, gc, i, table, lens)

        def both(i):
            store(i)
            paged(i)

        self.time("grouped", f"QK norm + rotary + store, {tag}", "", store, n, batch * (2 * H + 4 * Hkv) * D * 2)
        self.time("grouped", f"paged decode attention, {tag}", "", paged, n, g_bytes)
        self.time("grouped", f"store + decode attention, {tag}", "", both, n, g_bytes)

    def prefill_attention(self, tokens: int) -> None:
        from prism_infer_b200 import ops
        from prism_infer_b200.ops import latent as lat

        H, D, R, dev = self.heads, self.dim, self.rank, "cuda"
        cu = torch.tensor([0, tokens], dtype=torch.int32, device=dev)
        pages = -(-tokens // 256)
        table = torch.arange(pages, dtype=torch.int32, device=dev).view(1, -1)
        n = 2
        cache = ops.KVCache(n, pages, 1, 256, R, ops.KV_BF16, dev, planes=1)
        slots = torch.arange(tokens, device=dev)
        lws = [lat.LatentWeights(H, D, D, R, D ** -0.5, torch.ones(R, device=dev, dtype=torch.bfloat16), self.matrix(2 * H * D, R)) for _ in range(n)]
        q, raw, gate = self.matrix(tokens, H * D), self.matrix(tokens, R), self.matrix(tokens, H * D)
        core = 2.0 * tokens * tokens * H * D  # causal: half of 4 T^2 H D
        expand = 2.0 * tokens * R * 2 * H * D
        self.time("latent", f"latents -> keys, values -> gated attention, {tokens} tokens", "causal attention",
                  lambda i: lat.latent_attention_expanded(q, raw, gate, lws[i], 1e-5, slots, cache, i, table, cu, tokens), n, 0, core + expand)
        kv = self.matrix(tokens, 2 * H * D)
        from prism_infer_b200.ops import native

        out = torch.empty(tokens, H * D, device=dev, dtype=torch.bfloat16)

        def flash(_):
            native.call("prism_flash_attention_tc_kv", q.data_ptr(), q.stride(0), kv.data_ptr(), kv[:, H * D:].data_ptr(), kv.stride(0),
                        out.data_ptr(), out.stride(0), cu.data_ptr(), None, gate.data_ptr(), gate.stride(0), tokens, tokens, 1, tokens, H, H, D,
                        D ** -0.5, torch.cuda.current_stream().cuda_stream, ops._pdl())

        self.time("latent", f"gated causal attention, {tokens} tokens", "causal attention", flash, n, 0, core)
        c = self.matrix(tokens, R)
        self.time("latent", f"latents -> keys and values, {tokens} tokens", "gate/up projection", lambda i: ops.linear(c, lws[i].ukv), n,
                  2 * H * D * (R + tokens) * 2, expand)
        rows = torch.empty(tokens, R, device=dev, dtype=torch.bfloat16)
        self.time("latent", f"latent norm + store, {tokens} tokens", "QK norm + rotary + store",
                  lambda i: lat.latent_norm_store(raw, lws[i], 1e-5, slots, cache, i, rows=rows), n, tokens * R * 6)
        Hkv = H // 4
        q3, k3 = q.view(tokens, H, D), self.matrix(tokens, 2 * Hkv * D).view(tokens, 2 * Hkv, D)
        self.time("grouped", f"causal attention, {tokens} tokens", "", lambda _: ops.varlen_attention(q3, k3[:, :Hkv], k3[:, Hkv:], cu, tokens, causal=True),
                  n, 0, core)
        gc = ops.KVCache(n, pages, Hkv, 256, D, ops.KV_BF16, dev)
        qkv, one = self.matrix(tokens, (H + 2 * Hkv) * D), torch.ones(D, device=dev, dtype=torch.bfloat16)
        pos = torch.arange(tokens, dtype=torch.int32, device=dev).repeat(3, 1).contiguous()
        self.time("grouped", f"QK norm + rotary + store, {tokens} tokens", "", lambda i: ops.qk_norm_rope_store(
            qkv=qkv, partials=None, positions=pos, q_weight=one, k_weight=one, num_heads=H, num_kv_heads=Hkv, head_dim=D, theta=1e6,
            section=(24, 20, 20), eps=1e-6, slots=slots, cache=gc, layer=i), n, tokens * (2 * H + 4 * Hkv) * D * 2)


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
            k.projections(tokens)
            k.residual(tokens)
        for batch, context in ((1, 2048), (32, 2048), (128, 2048), (1, 16384)):
            k.decode_attention(batch, context)
            torch.cuda.empty_cache()
        for tokens in (2048, 8192):
            k.prefill_attention(tokens)
        rows += k.rows
        del k
        torch.cuda.empty_cache()
    return rows


def main(argv: list[str] | None = None) -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--sizes", default="2048,4096,8192")
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
    out = {"workload": "latent-layers", "data": "synthetic (random weights and token ids)", "dtype": "bf16",
           "l2": "operand sets or weights larger than L2", "models": models, "kernels": kernels, "clocks": sampler.stop()}
    text = json.dumps(out)
    if args.output:
        with open(args.output, "w", encoding="utf-8") as fh:
            fh.write(text + "\n")
    print(text)
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
