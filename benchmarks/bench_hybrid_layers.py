"""Prefill and decode throughput of the Fosulix family (gated linear attention, windowed latent attention with a rotated key part,
short convolutions, an average over the depth, bounded experts) beside the closest family, Bokorax, at equal layer sizes (random
weights), and every kernel of a layer against its roofline.

    python bench.py --workload hybrid-layers [--sizes 2048,4096] [--steps K] [--warmup W]
    python -m benchmarks.bench_hybrid_layers --kernels-only

Rows as in ``bench_latent_layers.py``; ``like`` names the row of the same size that a kernel is compared with.  Like kernels: the
state recurrence, blends, routing and windowed attention of Bokorax, the latent attention of Poralorn over as many keys.
"""

from __future__ import annotations

import argparse
import json
import sys

import torch

from benchmarks import bench_latent_layers as base
from benchmarks import bench_recurrent_layers as recurrent

LAYERS, VOCAB, WINDOW, TAPS = base.LAYERS, base.VOCAB, 1024, 4
STATE_DIM = recurrent.STATE_DIM
# width -> (heads, head width, rotated, latent, query latent, experts, chosen, expert feed-forward)
SIZES = {2048: (16, 128, 64, 256, 768, 32, 4, 768), 4096: (32, 128, 64, 512, 1536, 32, 4, 1536), 8192: (64, 128, 64, 512, 1536, 32, 4, 3072)}


def arch(width: int, kind: str):
    """``kind``: ``forget``, ``latent`` (layers of one mixer); ``recurrent``, ``windowed`` (the closest family's)."""
    from dataclasses import replace

    from prism_infer_b200.models.architecture import FosulixArch, ForgetMixArch, FosulixLayer, LatentAttentionArch, MixtureArch, RotaryArch

    H, D, r, R, Q, E, top, EF = SIZES[width]
    if kind in ("recurrent", "windowed"):
        a = recurrent.arch(width, kind)
        moe = MixtureArch(E, top, EF, scored=True, groups=4, groups_kept=2, scale=2.5)
        return replace(a, layers=tuple(replace(l, moe=moe) for l in a.layers))
    moe = MixtureArch(E, top, EF, scored=True, groups=4, groups_kept=2, scale=2.5, sigmoid=True, limit=7.0)
    rot = RotaryArch(1.0e6, r, factor=4.0, original=8192.0, fast=32.0, slow=1.0)
    mixer = (ForgetMixArch(width // STATE_DIM, STATE_DIM, STATE_DIM) if kind == "forget"
             else LatentAttentionArch(H, D, D, R, (D + r) ** -0.5, q_rank=Q, rot_dim=r, rot=rot, window=WINDOW))
    return FosulixArch(vocab_size=VOCAB, width=width, layers=(FosulixLayer(mixer, moe),) * LAYERS, taps=TAPS)


def model_rows(widths, batches, prompts, context: int, steps: int, warmup: int) -> list[dict]:
    rows = []
    for width in widths:
        for family in ("forget", "recurrent", "latent", "windowed"):
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
        self.H, self.D, self.r, self.R, self.Q, self.E, self.top, self.EF = SIZES[width]

    # ---- the forget rule and the convolution -----------------------------------------------------------
    def recurrence(self, tokens: int, batch: int = 1, dim: int = STATE_DIM) -> None:
        """``batch`` sequences of ``tokens`` each; one token: a decode step."""
        from prism_infer_b200.ops import latent as lat
        from prism_infer_b200.ops import native
        from prism_infer_b200.ops import recurrent as rec

        dev, W = "cuda", self.width
        H, T, decode = W // dim, tokens * batch, tokens == 1
        sp = rec.ForgetSpec(H, dim, dim, 1e-6)
        tag = (f"batch {batch}" if decode else f"{tokens} tokens" + (f" x {batch}" if batch > 1 else ""))
        tag = (f"heads of {dim}, " if dim != STATE_DIM else "") + tag
        like = (lambda name: f"{name}, {tag}") if dim == STATE_DIM else (lambda name: "")
        carry = (TAPS - 1) * W
        state_bytes = batch * sp.carry * 4
        sets = self.sets_for(2 * state_bytes if decode else 4 * sp.proj_cols * W * 2)
        cache = rec.StateCache([sp.carry + carry] * sets, batch, dev)
        slots = torch.arange(batch, dtype=torch.int32, device=dev)
        lens = torch.full((batch,), 64 + tokens, dtype=torch.int32, device=dev)
        cu = None if decode else (torch.arange(batch + 1, dtype=torch.int32, device=dev) * tokens)
        views = [rec.StateView(cache, i, slots, lens, cu) for i in range(sets)]
        ones = torch.ones(sp.gate_col, device=dev, dtype=torch.bfloat16)
        w = rec.ForgetWeights(2.0 * ones, 0.5 * ones, torch.ones(sp.m, device=dev, dtype=torch.bfloat16))
        small = T <= 128
        x = self.matrix(T, W)
        if dim == STATE_DIM:
            from prism_infer_b200.models.common import TPComm

            comm, n = TPComm(), self.sets_for(sp.proj_cols * W * 2)
            ws = [self.matrix(sp.proj_cols, W) for _ in range(n)]
            self.time("fosulix", f"stacked projection, {tag}", f"four projections, {tag}", lambda i: comm.row_parallel(x, ws[i]), n,
                      sp.proj_cols * W * 2 + T * (W * 2 + sp.proj_cols * (4 if small else 2)), 2.0 * sp.proj_cols * W * T)
            del ws
        p = lat.Branch(slabs=torch.randn(1, T, sp.proj_cols, device=dev)) if small else lat.Branch(rows=torch.randn(T, sp.proj_cols, device=dev, dtype=torch.bfloat16))
        p_bytes = T * sp.proj_cols * (4 if small else 2)
        if decode:
            self.time("fosulix", f"state step, {tag}", like("state step"), lambda i: rec.forget_mix(p, sp, w, views[i]), sets,
                      2 * state_bytes + p_bytes + T * H * sp.m * 2)
            return
        o, out = torch.empty(T, H * sp.m, device=dev), torch.empty(T, H * sp.m, device=dev, dtype=torch.bfloat16)
        st = lambda: torch.cuda.current_stream().cuda_stream  # noqa: E731

        def scan(i):
            native.call("prism_forget_scan", 0, *views[i].args(sp), batch, *rec._proj_args(p), w.bias.data_ptr(), w.lower.data_ptr(), o.data_ptr(), T,
                        H, sp.n, sp.m, st(), rec._pdl())

        self.time("fosulix", f"state scan, {tag}", like("state scan"), scan, min(sets, 8), p_bytes + T * H * sp.m * 4 + 2 * state_bytes,
                  5.0 * T * H * sp.n * sp.m, recurrent.FP32_RATE)
        self.time("fosulix", f"norm per head, {tag}", like("norm per head and gate"), lambda i: native.call(
            "prism_head_norm_gate", 0, o.data_ptr(), None, 0, 0, None, 0, w.norm.data_ptr(), out.data_ptr(), T, H, sp.m, sp.vdim, 1e-6, st(),
            rec._pdl()), 4, T * H * sp.m * 6)
        if dim == STATE_DIM:
            conv = rec.ConvSpec(TAPS, W, sp.carry)
            taps = self.matrix(TAPS, W)
            n = self.sets_for(T * W * 4)
            xs = [self.matrix(T, W) for _ in range(n)]
            self.time("fosulix", f"short convolution, {tag}", f"blends with the previous token, {tag}",
                      lambda i: rec.short_conv(xs[i], taps, conv, views[i % sets], max_len=tokens), n, T * W * 4)

    # ---- residual stream, router, experts ---------------------------------------------------------------
    def shared(self, tokens: int, depth: int = 3) -> None:
        from prism_infer_b200.ops import latent as lat
        from prism_infer_b200.ops import moe
        from prism_infer_b200.ops import recurrent as rec

        W, E, K, EF, tag, dev = self.width, self.E, self.top, self.EF, f"{tokens} tokens", "cuda"
        small = tokens <= 128
        x = self.matrix(tokens, W)
        router = [self.matrix(E, W) for _ in range(8)]
        self.time("fosulix", f"router logits, {tag}", f"router logits, {tag}", lambda i: lat.linear_slabs(x, router[i]), 8, E * W * 2 + tokens * (W * 2 + E * 4))
        slots, logits = torch.arange(tokens, device=dev), torch.randn(1, tokens, E, device=dev)
        zero = torch.zeros(E, device=dev)
        ours, theirs = moe.Scored(zero, 0, 4, 2, 2.5, sigmoid=True, group_best=2), moe.Scored(zero, 0, 4, 2, 2.5)
        for family, s in (("fosulix", ours), ("bokorax", theirs)):
            self.time(family, f"routing, {tag}", f"routing, {tag}" if family == "fosulix" else "",
                      lambda i: moe.route(lat.Branch(slabs=logits), K, E, 0, slots, scored=s), 4, tokens * E * 4)
        r = moe.route(lat.Branch(slabs=logits), K, E, 0, slots, scored=ours)
        used = int(r.n_groups[0]) if small else E
        n = max(2, min(4, self.sets_for(used * 3 * EF * W * 2)))
        gu, down = [self.matrix(E * 2 * EF, W).view(E, 2 * EF, W) for _ in range(n)], [self.matrix(E * W, EF).view(E, W, EF) for _ in range(n)]
        for family, act in (("fosulix", "bounded"), ("bokorax", "silu")):
            self.time(family, f"experts, {tag}", f"experts, {tag}" if family == "fosulix" else "",
                      lambda i: moe.expert_ffn(x, r, gu[i], down[i], act, 7.0), n, used * 3 * EF * W * 2 + tokens * K * (W * 6 + EF * 4), 6.0 * tokens * K * EF * W)
        del gu, down
        w = torch.ones(W, device=dev, dtype=torch.bfloat16)
        n = self.sets_for(tokens * W * (4 * depth + 16))
        data = [dict(x=torch.zeros(tokens, W, device=dev), n=self.matrix(tokens, W), h=torch.zeros(depth + 1, tokens, W, device=dev)) for _ in range(n)]
        ys = [torch.zeros(1, tokens * K, W, device=dev) if small else self.matrix(tokens * K, W) for _ in range(min(n, 8))]
        a = torch.ones(depth + 1, device=dev)
        branch = lambda i: lat.Branch(slabs=ys[i % len(ys)] if small else None, rows=None if small else ys[i % len(ys)], pos=r.pos, weight=r.weight)  # noqa: E731
        moved = tokens * K * W * (4 if small else 2) + tokens * W * (8 + 2)
        conv = carried = None
        if small:
            spec = rec.ConvSpec(TAPS, W, 0)
            cache = rec.StateCache([(TAPS - 1) * W] * n, tokens, dev)
            taps, lens = self.matrix(TAPS, W), torch.full((tokens,), 70, dtype=torch.int32, device=dev)
            conv = [rec.ConvStep(taps, spec, rec.StateView(cache, i, slots.to(torch.int32), lens)) for i in range(n)]
            carried = tokens * W * 8 * (TAPS - 1)

        def behind_layer(i):
            d = data[i]
            lat.stream_update(d["x"], W, 1e-5, keep=True, a=branch(i), mult=0.5, norm_weight=w, norm_out=d["n"], history=d["h"], depth=depth,
                              depth_weight=a, conv=conv[i] if conv else None)

        def plain(i, post=None):
            d = data[i]
            b = branch(i)
            b.post_norm = post
            lat.stream_update(d["x"], W, 1e-5, keep=True, a=b, mult=0.5, **({"raw_out": d["n"]} if post is not None else {"norm_weight": w, "norm_out": d["n"]}))

        self.time("fosulix", f"expert sum + average of {depth + 1} + norm" + (" + convolution" if conv else "") + f", {tag}", f"expert sum + norm + residual, {tag}",
                  behind_layer, n, moved + tokens * W * 4 * (depth + 1) + (carried or 0))
        self.time("fosulix", f"expert sum + residual + norm, {tag}", f"expert sum + norm + residual, {tag}", plain, n, moved)
        self.time("bokorax", f"expert sum + norm + residual, {tag}", "", lambda i: plain(i, w), n, moved)

    # ---- latent attention -------------------------------------------------------------------------------
    def latent_weights(self, sets: int):
        from prism_infer_b200.ops import latent as lat

        Rc = -(-(self.R + self.r) // 64) * 64
        rot = lat.Rotary(torch.rand(self.r // 2, device="cuda"), self.r, self.D, self.R)
        one = lambda n: torch.ones(n, device="cuda", dtype=torch.bfloat16)  # noqa: E731
        return Rc, [lat.LatentWeights(self.H, self.D + self.r, self.D, self.R, (self.D + self.r) ** -0.5, one(self.R), self.matrix(self.H * (2 * self.D + self.r), Rc),
                                      rot, WINDOW, self.Q, one(self.Q)) for _ in range(sets)]

    def projections(self, tokens: int) -> None:
        from prism_infer_b200.models.common import TPComm

        comm, tag, small, W = TPComm(), f"{tokens} tokens", tokens <= 128, self.width
        for family, name, m, k in (("fosulix", "latent projections", self.Q + self.R + self.r, W), ("fosulix", "query projection", self.H * (self.D + self.r), self.Q),
                                   ("fosulix", "attention output projection", W, self.H * self.D), ("bokorax", "stacked projection", (self.H + self.H // 2) * self.D, W)):
            x, n = self.matrix(tokens, k), self.sets_for(m * k * 2)
            ws = [self.matrix(m, k) for _ in range(n)]
            self.time(family, f"{name}, {tag}", "" if family == "bokorax" else f"stacked projection, {tag}", lambda i: comm.row_parallel(x, ws[i]), n,
                      m * k * 2 + tokens * (k * 2 + m * (4 if small else 2)), 2.0 * m * k * tokens)

    def decode_attention(self, batch: int, context: int) -> None:
        from prism_infer_b200 import ops
        from prism_infer_b200.ops import latent as lat
        from prism_infer_b200.ops import native

        H, D, r, R, Q, page, dev = self.H, self.D, self.r, self.R, self.Q, 256, "cuda"
        keys = min(context, WINDOW)
        per_seq = -(-context // page)
        lens = torch.full((batch,), context, dtype=torch.int32, device=dev)
        table = torch.randperm(batch * per_seq, device=dev).to(torch.int32).view(batch, per_seq)
        slots = table[:, -1].long() * page + (context - 1) % page
        pos = torch.full((batch,), context - 1, dtype=torch.int32, device=dev)
        Rc = -(-(R + r) // 64) * 64
        kv_bytes, u_bytes = batch * keys * (R + r) * 2, H * (2 * D + r) * Rc * 2
        n = self.sets_for(kv_bytes)
        Rc, lws = self.latent_weights(n)
        cache = ops.KVCache(n, batch * per_seq, 1, page, Rc, ops.KV_BF16, dev, planes=1)
        cache.payload.normal_()
        tag = f"batch {batch}, {keys} keys"
        splits = ops.choose_splits(Q + R + r, self.width, batch)
        y = lat.Branch(slabs=torch.randn(splits, batch, Q + R + r, device=dev))
        self.time("fosulix", f"latent norms + rotary + store, batch {batch}", f"prepare queries and cache rows (window, tied values), {batch} tokens",
                  lambda i: lat.latent_prepare(y, lws[i], 1e-6, pos, slots, cache, i), n, batch * (Q + R + r) * (4 * splits + 2))
        qs = ops.choose_splits(H * (D + r), Q, batch)
        q = lat.Branch(slabs=torch.randn(ops.effective_splits(Q, qs), batch, H * (D + r), device=dev))
        ns = lat.latent_splits(batch, H, WINDOW + 1)
        qa = torch.randn(batch, H, Rc, device=dev, dtype=torch.bfloat16)
        po = torch.empty(batch * H, ns, R, device=dev) if ns > 1 else None
        ml = torch.zeros(batch * H, ns, 2, device=dev) if ns > 1 else None
        la = torch.empty(batch * H, R, device=dev, dtype=torch.bfloat16)
        out = torch.empty(batch, H * D, device=dev, dtype=torch.bfloat16)
        p, s, pdl = (lambda t: None if t is None else t.data_ptr()), (lambda: torch.cuda.current_stream().cuda_stream), ops._pdl

        def absorb(i):
            l, src, rot = lws[i], q, (*lws[i].rot.args(pos), D, r)
            if batch > lat.ABSORB_ROTATES_TOKENS:
                src, rot = lat.Branch(rows=lat.rotate_queries(q, l, pos)), (*lat.NO_ROTARY, 0, 0)
            slabs, stride, P, rows, ld = lat._branch_args(src)
            native.call("prism_latent_absorb", rows, slabs, stride, P, ld, *rot, p(l.uk), p(qa), None, 0, None, None, p(slots), 0, batch, H, D + r,
                        R, Rc, 1e-6, s(), pdl())

        def attend(i):
            native.call("prism_latent_attention", p(qa), p(cache.latent(i)), p(table), None, p(lens), p(po), p(ml), p(la), batch, 1, H, Rc, R, page, per_seq,
                        cache.num_blocks, ns, WINDOW, (D + r) ** -0.5, s(), pdl())

        def output(i):
            native.call("prism_latent_out", p(po), p(ml), p(la), p(lws[i].uv), Rc, None, 0, p(out), out.stride(0), batch, H, D, R, ns, s(), pdl())

        self.time("fosulix", f"rotary + absorb, batch {batch}", f"absorb + latent store, {tag}", absorb, n,
                  H * (D + r) * Rc * 2 + batch * H * ((D + r) * 4 * q.slabs.shape[0] + Rc * 2))
        self.time("fosulix", f"latent attention in a window, {tag}", f"latent attention, {tag}", attend, n, kv_bytes + batch * H * (R + Rc) * 2,
                  2.0 * batch * H * keys * (2 * R + r))
        self.time("fosulix", f"merge + value up, {tag}", f"merge + value up + gate, {tag}", output, n, H * D * R * 2 + batch * H * (R + D) * 2)
        del u_bytes

    def prefill_attention(self, tokens: int) -> None:
        from prism_infer_b200 import ops
        from prism_infer_b200.ops import latent as lat
        from prism_infer_b200.ops import native, window

        H, D, r, R, Q, page, dev = self.H, self.D, self.r, self.R, self.Q, 256, "cuda"
        cu = torch.tensor([0, tokens], dtype=torch.int32, device=dev)
        lens = torch.tensor([tokens], dtype=torch.int32, device=dev)
        pages = -(-tokens // page)
        table = torch.arange(pages, dtype=torch.int32, device=dev).view(1, -1)
        slots, pos = torch.arange(tokens, device=dev), torch.arange(tokens, dtype=torch.int32, device=dev)
        Rc, lws = self.latent_weights(2)
        cache = ops.KVCache(2, pages, 1, page, Rc, ops.KV_BF16, dev, planes=1)
        cache.payload.normal_()
        w = min(WINDOW, tokens)
        pairs = tokens * w - w * (w - 1) / 2
        tag = f"{tokens} tokens"
        y = lat.Branch(rows=self.matrix(tokens, Q + R + r))
        self.time("fosulix", f"latent norms + rotary + store, {tag}", f"prepare queries and cache rows (window, tied values), {tag}",
                  lambda i: lat.latent_prepare(y, lws[i], 1e-6, pos, slots, cache, i), 2, tokens * (Q + R + r) * 4)
        q = self.matrix(tokens, H * (D + r))
        self.time("fosulix", f"rotary of queries, {tag}", f"prepare queries and cache rows (window, tied values), {tag}",
                  lambda i: lat.rotate_queries(lat.Branch(rows=q), lws[i], pos), 2, tokens * H * r * 4)
        plan = lat.ExpandPlan.make([(tokens, tokens)], WINDOW, page, pages, dev)
        rows = torch.empty(plan.pages * page, Rc, device=dev, dtype=torch.bfloat16)

        def gather(i):
            native.call("prism_gather_latent_pages", cache.latent(i).data_ptr(), table.data_ptr(), lens.data_ptr(), plan.first.data_ptr(), plan.base.data_ptr(),
                        rows.data_ptr(), 1, plan.max_pages, rows.shape[0], pages, cache.num_blocks, page, Rc * 2, torch.cuda.current_stream().cuda_stream, ops._pdl())

        self.time("fosulix", f"visible rows gathered, {tag}", "", gather, 2, tokens * Rc * 4)
        M = H * (2 * D + r)
        self.time("fosulix", f"rows -> keys and values, {tag}", f"latents -> keys and values, {tag}", lambda i: ops.linear(rows, lws[i].ukv), 2,
                  M * (Rc + tokens) * 2, 2.0 * tokens * Rc * M)
        kv = lat._ScratchPages(self.matrix(tokens, M).view(pages, page, M))
        sp = window.WindowSpec(heads=H, kv_heads=H, maps=1, dim=D + r, vdim=D, rot_dims=0, scale=(D + r) ** -0.5, window=WINDOW, keep_first=0, gate=False, eps=0.0)
        self.time("fosulix", f"windowed attention of explicit keys, {tag}", f"prefill attention (window, tied values), {tag}",
                  lambda i: window.window_attention(q, sp, None, kv, 0, table, lens, cu_seqlens_q=cu, max_q_len=tokens), 2, 0, 2.0 * pairs * H * (2 * D + r))
        self.time("fosulix", f"all of the attention, {tag}", f"prefill attention (window, tied values), {tag}",
                  lambda i: lat.latent_attention_windowed(q, lws[i], cache, i, table, lens, cu, tokens, plan), 2, 0,
                  2.0 * pairs * H * (2 * D + r) + 2.0 * tokens * Rc * M)


def kernel_rows(widths, steps: int, warmup: int) -> list[dict]:
    from prism_infer_b200 import ops
    from prism_infer_b200.ops import native

    native.lib()
    ops.set_pdl(True)
    ops.apply_tuning()
    rows = []
    for width in widths:
        k, like, latent = Kernels(width, steps, warmup), recurrent.Kernels(width, steps, warmup), base.Kernels(width, steps, warmup)
        for tokens, batch in ((1, 1), (1, 32), (1, 128), (2048, 1), (8192, 1), (2048, 4)):
            k.recurrence(tokens, batch)
            like.recurrence(tokens, batch)
            k.recurrence(tokens, batch, 128)
            torch.cuda.empty_cache()
        for tokens in (1, 32, 128, 2048):
            k.shared(tokens)
            k.projections(tokens)
            torch.cuda.empty_cache()
        for tokens in (1, 32, 2048):
            like.shared(tokens)
            torch.cuda.empty_cache()
        for batch in (1, 32, 128):
            k.decode_attention(batch, 2048)
            latent.decode_attention(batch, WINDOW)
            like.decode_attention(batch, 2048)
            torch.cuda.empty_cache()
        for tokens in (2048, 8192):
            k.prefill_attention(tokens)
            like.prefill_attention(tokens)
            latent.prefill_attention(tokens)
            torch.cuda.empty_cache()
        rows += k.rows + like.rows + [r for r in latent.rows if r["family"] == "latent"]
        del k, like, latent
        torch.cuda.empty_cache()
    native.check_status()
    return rows


def compare(rows: list[dict]) -> list[dict]:
    """Every row with a like kernel: how many times further from its roofline, and the ratio of the times."""
    out = []
    for r in rows:
        if r["family"] != "fosulix" or not r["like"]:
            continue
        like = next((o for o in rows if o["width"] == r["width"] and o["kernel"] == r["like"] and o["family"] != "fosulix"), None)
        if like is not None:
            out.append({**r, "like_us": like["us"], "like_fraction": like["fraction"], "further": round(like["fraction"] / max(r["fraction"], 1e-6), 2),
                        "time_ratio": round(r["us"] / like["us"], 2)})
    return out


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
    out = {"workload": "hybrid-layers", "data": "synthetic (random weights and token ids)", "dtype": "bf16", "window": WINDOW,
           "l2": "operand sets or weights larger than L2", "models": models, "kernels": kernels, "beside": compare(kernels), "clocks": sampler.stop()}
    text = json.dumps(out)
    if args.output:
        with open(args.output, "w", encoding="utf-8") as fh:
            fh.write(text + "\n")
    print(text)
    return 0


if __name__ == "__main__":
    sys.exit(main())
