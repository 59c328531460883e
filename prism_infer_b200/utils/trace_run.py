"""Trace runner: feeds given token ids through a model, step by step, and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps are JSON objects, one a line, on standard input:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

An entry brings a request's next tokens and the places among them whose logits are wanted; ``end`` lists the requests
that are finished after the step.  Wanted logits go to ``OUT/<step>.f32`` (little-endian fp32 ``[wanted, vocab]``, in
the order of the entries), and every step is answered by a line ``done <step>``.  At most four requests are live at
a time and they hold at most ``--max-tokens`` tokens, each request's count rounded up to whole pages of 64.  Kernels
that have not been compiled yet are compiled at start-up.  Exit code 3: no 32-bit kernels for this model.
"""

from __future__ import annotations

import argparse
import json
import os
import sys

PAGE = 64
MAX_LIVE = 4


def build_parser() -> argparse.ArgumentParser:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay token ids through a model and write logits")
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True)
    ap.add_argument("--device", default="cuda:0", help="cpu: the engine's PyTorch statements of its ops (float32 only)")
    return ap


def main(argv: list[str] | None = None) -> int:
    args = build_parser().parse_args(argv)
    with open(os.path.join(args.model, "config.json"), "r", encoding="utf-8") as fh:
        config = json.load(fh)
    from ..models.model_registry import family_of_config

    family = family_of_config(config)
    on_cuda = args.device.startswith("cuda")
    if args.dtype == "float32" and on_cuda and not family.float32_on_cuda:
        print(f"trace_run: the {family.name} family has no 32-bit kernels", file=sys.stderr)
        return 3
    if on_cuda:
        from ..ops import build, native

        native.use_library(build.ensure(family.name, family.kernel_units) if family.kernel_units else build.build())
    from ..engine.llm_engine import LLMEngine
    from ..engine.replay import ReplayEntry, TraceReplay

    pages = max(1, -(-args.max_tokens // PAGE))
    engine = LLMEngine(args.model, device=args.device, dtype=args.dtype, max_model_len=pages * PAGE, kvcache_block_size=PAGE,
                       num_kvcache_blocks=pages, cpu_kv_cache_ratio=0.0, enable_prefix_caching=False, max_num_seqs=MAX_LIVE,
                       max_chunk_size=pages * PAGE, max_num_batched_tokens=max(16384, pages * PAGE), enable_step_logits=True,
                       enable_decode_run_ahead=False, enforce_eager=not on_cuda)
    replay = TraceReplay(engine)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = [ReplayEntry(e["id"], e["tokens"], e.get("want", ())) for e in step.get("entries", [])]
        logits = replay.step(entries, step.get("end", ()))
        if logits.shape[0]:
            logits.numpy().astype("<f4").tofile(os.path.join(args.out, f"{step['step']}.f32"))
        print(f"done {step['step']}", flush=True)
    if on_cuda:
        engine.check_device_status()
    engine.exit()
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
