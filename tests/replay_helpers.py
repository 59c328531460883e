"""Checkpoints, engines and replays of small text-only models, shared by the tests of the model families."""

import torch


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(1000 + seed)).tolist()


# ------------------------------------------------------------------------------------ engines and replays
def checkpoint(directory, arch, weights):
    """A checkpoint directory as a user would have it: config.json and bf16 safetensors."""
    from prism_infer_b200.models.weights import save_checkpoint

    save_checkpoint(str(directory), arch, {k: v.to(torch.bfloat16) for k, v in weights.items()})
    return str(directory)


def engine(path, backend, **kw):
    from prism_infer_b200 import LLM

    device, dtype = backend
    options = dict(max_model_len=640, kvcache_block_size=16, num_kvcache_blocks=48, cpu_kv_cache_ratio=0.0, max_num_seqs=4,
                   enable_prefix_caching=False, enable_step_logits=True, enable_decode_run_ahead=False, dtype=dtype,
                   enforce_eager=not device.startswith("cuda"), max_chunk_size=640, max_num_batched_tokens=1024)
    options.update(kw)
    return LLM(path, device=device, **options)


def replay(llm, steps):
    """``steps``: lists of (request, tokens); a request whose name ends a step's ``end`` set gives its pages back.
    Returns request -> logits of every token fed, in order."""
    from prism_infer_b200.engine.replay import ReplayEntry, TraceReplay

    session = TraceReplay(llm)
    out = {}
    for entries, end in steps:
        logits = session.step([ReplayEntry(r, t, range(len(t))) for r, t in entries], end)
        base = 0
        for r, t in entries:
            out.setdefault(r, []).append(logits[base:base + len(t)])
            base += len(t)
    return {r: torch.cat(parts) for r, parts in out.items()}


def portions(request, toks, sizes):
    """Steps that feed ``toks`` in portions of the given sizes, cycled; the request ends with its last portion."""
    steps, at, i = [], 0, 0
    while at < len(toks):
        n = sizes[i % len(sizes)]
        part = toks[at:at + n]
        at, i = at + len(part), i + 1
        steps.append(([(request, part)], [request] if at == len(toks) else []))
    return steps


def error(got, want):
    """Largest over the positions of the root mean square difference, relative to the spread of the logits."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt() / want.double().std()).max())
