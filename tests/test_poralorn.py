"""The Poralorn family through the engine (configuration, loading, paged latents, portions, mixed batches, greedy
generation) against the plain statement in ``poralorn_oracle.py``: on the CPU in 32-bit, on a B200 in 32-bit and bf16."""

import gc
import json
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import poralorn_cases as cases  # noqa: E402
import poralorn_oracle as oracle  # noqa: E402

from prism_infer_b200 import LLM, SamplingParams  # noqa: E402
from prism_infer_b200.config import Config  # noqa: E402
from prism_infer_b200.models.architecture import PoralornArch  # noqa: E402
from prism_infer_b200.models.model_registry import family_of_config  # noqa: E402

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
CPU = ("cpu", "float32")
GPU32 = pytest.param(("cuda:0", "float32"), marks=pytest.mark.gpu, id="gpu-float32")
GPU16 = pytest.param(("cuda:0", "bfloat16"), marks=pytest.mark.gpu, id="gpu-bfloat16")
BACKENDS = [pytest.param(CPU, id="cpu"), GPU32, GPU16]
LIMIT = {"float32": 2e-5, "bfloat16": 0.03}


@pytest.fixture(scope="module")
def model(tmp_path_factory):
    """name -> (config, architecture, weights, checkpoint directory), built once."""
    made = {}

    def get(name):
        if name not in made:
            cfg, arch, w = cases.make(name)
            made[name] = (cfg, arch, w, cases.checkpoint(tmp_path_factory.mktemp(name), arch, w))
        return made[name]

    return get


# ---------------------------------------------------------------------------------- configuration and loading
def test_config_round_trip_and_layer_runs():
    for name, cfg in cases.CASES.items():
        arch = PoralornArch.from_hf_config(cfg)
        assert family_of_config(cfg).name == "poralorn"
        assert PoralornArch.from_hf_config(json.loads(json.dumps(arch.to_hf_config()))) == arch, name
    runs = PoralornArch.from_hf_config(cases.CASES["uneven"]).layer_runs()
    assert [(r.layer, r.loop_pass) for r in runs] == [(0, None), (1, 0), (2, None), (1, 1), (2, None)]
    assert [(r.layer, r.loop_pass) for r in PoralornArch.from_hf_config(cases.CASES["once"]).layer_runs()] == [(0, 0)]
    assert [(r.layer, r.loop_pass) for r in PoralornArch.from_hf_config(cases.CASES["wide"]).layer_runs()] == [(0, None), (1, None)]


def test_config_is_checked():
    good = cases.CASES["tail"]
    for change in ({"layers": []}, {"loop": {"start": 2, "stop": 2, "times": 1}}, {"loop": {"start": 0, "stop": 9, "times": 1}},
                   {"layers": [{**good["layers"][0], "type": "other"}]}, {"layers": [{**good["layers"][0], "mlp": {"kind": "x", "ff": 8}}]}):
        with pytest.raises(ValueError):
            PoralornArch.from_hf_config({**good, **change})
    for missing in ("vocab", "width", "norm", "residual_mult", "layers"):
        with pytest.raises(ValueError, match=missing):
            PoralornArch.from_hf_config({k: v for k, v in good.items() if k != missing})


def test_options_the_family_does_not_have_are_refused():
    for kw in ({"compression_mode": "scaled_fp8_kv"}, {"compression_mode": "visual_compact"}, {"tensor_parallel_size": 2}):
        with pytest.raises(ValueError):
            Config("random:poralorn-tiny", **kw)
    llm = LLM("random:poralorn-tiny", device="cpu", enforce_eager=True, kvcache_block_size=16, num_kvcache_blocks=4, max_model_len=64)
    with pytest.raises(ValueError, match="text"):
        llm.generate_images("1 2", [])
    with pytest.raises(ValueError):
        LLM("random:poralorn-tiny", device="cpu", dtype="bfloat16")


def test_loading_checks_names_and_shapes(model):
    cfg, arch, w, _ = model("uneven")
    from prism_infer_b200.models.poralorn import PoralornModel

    m = PoralornModel(arch, device="cpu", dtype=torch.float32)
    with pytest.raises(KeyError, match="missing"):
        m.load((k, v) for k, v in w.items() if k != "l1.rg1.b")
    with pytest.raises(ValueError, match="loop.in"):
        m.load({**w, "loop.in": w["loop.in"][:, :-1]}.items())
    m.load({**w, "unknown.tensor": torch.zeros(3)}.items())


def test_environment_check_knows_the_family(model):
    from prism_infer_b200.utils.check_environment import inspect_checkpoint

    rep, errors, _ = inspect_checkpoint(model("uneven")[3], 1)
    assert rep["status"] == "pass" and not errors and rep["text"]["layer_runs"] == 5
    assert inspect_checkpoint(model("uneven")[3], 2)[1]


def test_partial_kernel_library(tmp_path, monkeypatch):
    """Without an up-to-date full library only the family's own kernel units are compiled, into a library of their own."""
    from prism_infer_b200.models.model_registry import resolve_model_family
    from prism_infer_b200.ops import build

    units = resolve_model_family("poralorn").kernel_units
    assert {u + ".cu" for u in units} <= set(build._sources())
    asked = {}
    monkeypatch.setattr(build, "build", lambda **kw: asked.update(kw) or kw["target"])
    monkeypatch.setattr(build, "BUILD", str(tmp_path))
    monkeypatch.setattr(build, "LIB", str(tmp_path / "absent.so"))
    assert build.ensure("poralorn", units) == build.partial_library("poralorn") and asked["units"] == units


def test_cache_geometry():
    arch = PoralornArch.from_hf_config(cases.CASES["uneven"])
    g = arch.kv_geometry()
    assert (g.planes, g.layers, g.heads, g.row) == (1, 5, 1, 192)
    assert g.bytes_per_page(64, 2) == 5 * 64 * 192 * 2
    assert Config("random:poralorn-tiny", kvcache_block_size=64).kv_bytes_per_page() == PoralornArch.tiny().num_layer_runs * 64 * 128 * 2


# ----------------------------------------------------------------------------------------- whole forward
@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", list(cases.CASES))
def test_whole_prompt_and_residual_stream(model, name, backend):
    """Logits at every position, and the stream after every layer run."""
    cfg, arch, w, path = model(name)
    toks = cases.tokens(83, arch.vocab_size)
    want, states = oracle.forward(toks, w, cfg)
    llm = cases.engine(path, backend)
    got = cases.replay(llm, [([("a", toks)], ["a"])])["a"]
    assert cases.error(got, want) < LIMIT[backend[1]]
    runner = llm.runners.runner
    from prism_infer_b200.models.common import AttnMeta

    dev, n = runner.device, len(toks)
    table = torch.arange(6, dtype=torch.int32).view(1, -1).to(dev)
    meta = AttnMeta(is_prefill=True, block_tables=table, slots=torch.arange(n).to(dev), max_q_len=n, no_history=True, total_kv=n,
                    max_kv_len=n, attended_pairs=n * n, cu_seqlens_q=torch.tensor([0, n], dtype=torch.int32).to(dev),
                    kv_lens=torch.tensor([n], dtype=torch.int32).to(dev))
    st = runner.model.begin_layers(torch.tensor(toks).to(dev), torch.zeros((3, n), dtype=torch.int32).to(dev), meta, runner.kv)
    for i in range(arch.num_layer_runs):
        runner.model.advance_layers(st, 1)
        x = st.x.double().cpu()
        assert bool((x[:, arch.width:] == 0).all())
        d = (x[:, :arch.width] - states[i]).abs().max() / states[i].abs().max()
        assert float(d) < (1e-5 if backend[1] == "float32" else 0.03), i
    llm.exit()


@pytest.mark.parametrize("backend", BACKENDS)
def test_first_tokens_of_a_sequence(model, backend):
    cfg, arch, w, path = model("uneven")
    llm = cases.engine(path, backend)
    for n in (1, 2, 3, 15, 16, 17):
        toks = cases.tokens(n, arch.vocab_size, seed=n)
        got = cases.replay(llm, [([("a", toks)], ["a"])])["a"]
        assert cases.error(got, oracle.forward(toks, w, cfg)[0]) < LIMIT[backend[1]], n
    llm.exit()


# ---------------------------------------------------------------------- decoding, portions, batches, pages
@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", ["uneven", "ragged", "wide"])
def test_token_by_token_decoding_equals_the_prompt(model, name, backend):
    cfg, arch, w, path = model(name)
    toks = cases.tokens(70, arch.vocab_size, seed=3)
    want, _ = oracle.forward(toks, w, cfg)
    llm = cases.engine(path, backend)
    got = cases.replay(llm, cases.portions("a", toks, [1]))["a"]
    assert cases.error(got, want) < LIMIT[backend[1]]
    llm.exit()


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("sizes", [[2], [3, 37, 1], [16], [15, 17], [64, 5], [1, 2, 90]])
def test_portions_of_a_prompt(model, sizes, backend):
    cfg, arch, w, path = model("tail")
    toks = cases.tokens(150, arch.vocab_size, seed=5)
    want, _ = oracle.forward(toks, w, cfg)
    llm = cases.engine(path, backend)
    got = cases.replay(llm, cases.portions("a", toks, sizes))["a"]
    assert cases.error(got, want) < LIMIT[backend[1]]
    llm.exit()


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", ["uneven", "tail"])
def test_mixed_batches_and_reused_pages(model, name, backend):
    """Portions of some requests beside single tokens of others, requests left out of steps, pages freed and used
    again by later requests; a pool that holds exactly what is live."""
    cfg, arch, w, path = model(name)
    t = {r: cases.tokens(n, arch.vocab_size, seed=i) for i, (r, n) in enumerate({"a": 61, "b": 34, "c": 130, "d": 20, "e": 97}.items())}
    at = {r: 0 for r in t}

    def take(r, n):
        part = t[r][at[r]:at[r] + n]
        at[r] += len(part)
        return r, part

    steps = [([take("a", 30), take("b", 2)], []), ([take("a", 1), take("b", 15), take("c", 64)], []), ([take("c", 2), take("a", 1)], []),
             ([take("a", 1), take("b", 1), take("c", 1)], []), ([take("b", 16), take("a", 1)], ["b"]),
             ([take("d", 20), take("c", 33), take("a", 1)], ["d"]), ([take("e", 80), take("a", 26), take("c", 1)], ["a"])]
    while at["c"] < len(t["c"]) or at["e"] < len(t["e"]):
        entries = [take(r, n) for r, n in (("c", 1), ("e", 1)) if at[r] < len(t[r])]
        steps.append((entries, [r for r, _ in entries if at[r] == len(t[r])]))
    llm = cases.engine(path, backend, num_kvcache_blocks=17)
    free = llm.scheduler.block_manager.gpu.num_free
    for repeat in range(2):  # the second time over other pages, with the first run's latents still in them
        got = cases.replay(llm, steps)
        for r in t:
            assert cases.error(got[r], oracle.forward(t[r], w, cfg)[0]) < LIMIT[backend[1]], (r, repeat)
        assert llm.scheduler.block_manager.gpu.num_free == free
    llm.exit()


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("page", [16, 64])
def test_sharp_attention_finds_far_keys(tmp_path, backend, page):
    """Scores scaled up until each query looks at about one key, wherever it is: a wrong, lost or shifted key changes
    the output completely.  Positions around every page border, in a prompt, in portions and decoded."""
    mix = cases.mixer(3, 32, 32, 64, 1.6)
    cfg = cases.config([(mix, 48), (mix, 0)], vocab=150, width=96, loop=(0, 1, 2), mult=0.8)
    arch = PoralornArch.from_hf_config(cfg)
    from prism_infer_b200.models.weights import random_weights

    w = {k: (v * (1.0 if arch.init_kind(k) != "embedding" else 20.0)).to(torch.bfloat16).float() for k, v in random_weights(arch, seed=4).items()}
    path = cases.checkpoint(tmp_path, arch, w)
    toks = cases.tokens(270, arch.vocab_size, seed=9)
    want, _ = oracle.forward(toks, w, cfg)
    llm = cases.engine(path, backend, kvcache_block_size=page, num_kvcache_blocks=640 // page)
    whole = cases.replay(llm, [([("a", toks)], ["a"])])["a"]
    parts = cases.replay(llm, cases.portions("a", toks, [63, 2, 64, 1, 16]))["a"]
    decoded = cases.replay(llm, [([("a", toks[:190])], [])] + cases.portions("a", toks[190:], [1]))["a"]
    # rounding moves a score that decides between two keys: most positions, in 16 bits, and all of them in 32
    for got in (whole, parts, decoded):
        d = (got.double() - want)
        e = d.pow(2).mean(-1).sqrt() / want.std()
        assert float(e.quantile(0.9)) < (2e-4 if backend[1] == "float32" else 0.25)
        assert float(e.max()) < (2e-3 if backend[1] == "float32" else 1.2)
    llm.exit()


@pytest.mark.parametrize("backend", BACKENDS)
def test_long_decoding(model, backend):
    cfg, arch, w, path = model("once")
    toks = cases.tokens(300, arch.vocab_size, seed=11)
    want, _ = oracle.forward(toks, w, cfg)
    llm = cases.engine(path, backend)
    got = cases.replay(llm, [([("a", toks[:9])], [])] + cases.portions("a", toks[9:], [1]))["a"]
    assert cases.error(got, want) < LIMIT[backend[1]]
    llm.exit()


def test_replay_checks_its_input(model):
    from prism_infer_b200.engine.block_pool import OutOfBlocks
    from prism_infer_b200.engine.replay import ReplayEntry, TraceReplay

    _, arch, _, path = model("once")
    llm = cases.engine(path, CPU, num_kvcache_blocks=2, max_model_len=32)
    session = TraceReplay(llm)
    for entries in ([ReplayEntry("a", [])], [ReplayEntry("a", [arch.vocab_size])], [ReplayEntry("a", [1]), ReplayEntry("a", [2])]):
        with pytest.raises(ValueError):
            TraceReplay(llm).step(entries)
    with pytest.raises(OutOfBlocks):
        session.step([ReplayEntry("a", [1] * 17), ReplayEntry("b", [1])])
    cached = cases.engine(path, CPU, enable_prefix_caching=True)
    with pytest.raises(ValueError, match="prefix"):
        TraceReplay(cached)


# --------------------------------------------------------------------- the engine's entry point and scheduler
def _greedy_ok(got, prompt, w, cfg, slack):
    """Every generated token is the plain statement's arg-max, or as good as it to within ``slack`` logits."""
    logits, _ = oracle.forward(list(prompt) + list(got), w, cfg)
    for i, t in enumerate(got):
        row = logits[len(prompt) - 1 + i]
        assert float(row.max() - row[t]) <= slack, (i, float(row.max() - row[t]))


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("options", [
    {}, {"enable_prefix_caching": True, "enable_decode_run_ahead": True}, {"max_chunk_size": 24, "max_num_batched_tokens": 64},
    {"num_kvcache_blocks": 16, "cpu_kv_cache_ratio": 2.0}, {"num_kvcache_blocks": 16},
    {"enable_cooperative_prefill": True, "cooperative_prefill_layer_quantum": 1, "max_num_seqs": 2}],
    ids=["plain", "prefix-cache", "chunked", "swap", "recompute", "cooperative"])
def test_greedy_generation(model, options, backend):
    cfg, arch, w, path = model("uneven")
    shared = cases.tokens(48, arch.vocab_size, seed=30)
    prompts = [shared + cases.tokens(n, arch.vocab_size, seed=40 + n) for n in (1, 9, 30)] + [cases.tokens(5, arch.vocab_size, seed=50)]
    llm = cases.engine(path, backend, **options)
    sp = SamplingParams(temperature=0.0, max_tokens=20, ignore_eos=False)
    out = llm.generate(prompts, sp, use_tqdm=False)
    if options.get("enable_prefix_caching"):
        out = llm.generate(prompts, sp, use_tqdm=False)  # pages of the first round are hit
    for p, o in zip(prompts, out):
        assert len(o["token_ids"]) == 20
        _greedy_ok(o["token_ids"], p, w, cfg, 1e-3 if backend[1] == "float32" else 0.25)
    counters = llm.scheduler.counters
    if "cpu_kv_cache_ratio" in options:
        assert counters["preempt_swap"] > 0 and counters["swap_in"] > 0
    elif options.get("num_kvcache_blocks") == 16:
        assert counters["preempt_recompute"] > 0
    if backend[0] != "cpu":
        llm.check_device_status()
        assert llm.graph_metadata()["decode_steps"]["graph_batch_sizes"]
    llm.exit()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["auto", "float32"])
def test_cache_sized_from_free_memory(cuda_device, dtype):
    """Default cache sizing (a measured warm-up prefill) and graph decode on production widths."""
    llm = LLM("random:poralorn-8b-like-4layer" if dtype == "auto" else "random:poralorn-tiny", dtype=dtype, gpu_memory_utilization=0.3,
              max_num_seqs=8, max_num_batched_tokens=2048, cpu_kv_cache_ratio=0.0)
    sizing = llm.graph_metadata()["kv_sizing"]
    assert sizing["budget_bytes"] > 0 and llm.scheduler.block_manager.gpu.num_blocks > 100
    prompts = [cases.tokens(n, 200, seed=n) for n in (700, 3, 41)]
    together = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True), use_tqdm=False)
    assert all(len(o["token_ids"]) == 6 for o in together)
    llm.check_device_status()
    llm.exit()
    del llm
    gc.collect()  # the cache takes a third of the device: give it back before the next test
    torch.cuda.empty_cache()


@pytest.mark.parametrize("backend", BACKENDS)
def test_sampling_follows_the_capped_logits(model, backend):
    cfg, arch, w, path = model("once")
    prompt = cases.tokens(12, arch.vocab_size, seed=2)
    llm = cases.engine(path, backend)
    sp = SamplingParams(temperature=0.05, max_tokens=1, ignore_eos=True)
    drawn = [llm.generate([prompt], sp, use_tqdm=False)[0]["token_ids"][0] for _ in range(8)]
    row = oracle.forward(prompt, w, cfg)[0][-1]
    assert all(float(row.max() - row[t]) < 1.0 for t in drawn)  # 20 temperatures below the best
    llm.exit()


@pytest.mark.parametrize("backend", BACKENDS)
def test_served_over_http(model, backend):
    """The serving runtime answers text requests with the same greedy tokens and refuses media."""
    import asyncio

    import httpx

    from prism_infer_b200.serving.app import create_app
    from prism_infer_b200.serving.runtime import ServingRuntime

    cfg, arch, w, path = model("once")
    prompt = cases.tokens(10, arch.vocab_size, seed=6)
    runtime = ServingRuntime(lambda: cases.engine(path, backend))
    runtime.start()
    app = create_app(runtime, model_name="poralorn", manage_runtime=False)

    async def scenario():
        async with httpx.AsyncClient(transport=httpx.ASGITransport(app=app), base_url="http://t", timeout=60.0) as client:
            r = await client.post("/v1/generate", json={"prompt": " ".join(map(str, prompt)), "sampling": {"max_tokens": 6, "ignore_eos": True}})
            assert r.status_code == 200, r.text
            _greedy_ok(r.json()["token_ids"], prompt, w, cfg, 1e-3 if backend[1] == "float32" else 0.25)

    try:
        asyncio.run(scenario())
    finally:
        runtime.stop()


# ----------------------------------------------------------------------------------------- trace runner
def _run_trace(path, out, dtype, device, lines, max_tokens=256):
    cmd = [os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(out), "--max-tokens", str(max_tokens),
           "--device", device]
    return subprocess.run(cmd, input="".join(json.dumps(x) + "\n" for x in lines), capture_output=True, text=True, timeout=240)


@pytest.mark.parametrize("backend", BACKENDS)
def test_trace_runner(model, tmp_path, backend):
    cfg, arch, w, path = model("ragged")
    a, b = cases.tokens(70, arch.vocab_size, seed=1), cases.tokens(9, arch.vocab_size, seed=2)
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": a[:66], "want": [0, 63, 64, 65]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[:8], "want": []}, {"id": "a", "tokens": a[66:67], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[8:], "want": [0]}, {"id": "a", "tokens": a[67:68], "want": [0]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": a[68:], "want": [1]}], "end": ["a"]}]
    res = _run_trace(path, tmp_path, backend[1], backend[0], lines)
    assert res.returncode == 0, res.stderr
    assert [x for x in res.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    assert not (tmp_path / "1.f32").exists()
    wa, wb = oracle.forward(a, w, cfg)[0], oracle.forward(b, w, cfg)[0]

    def read(step):
        return torch.frombuffer(bytearray((tmp_path / f"{step}.f32").read_bytes()), dtype=torch.float32).view(-1, arch.vocab_size)

    for got, want in ((read(0), wa[[0, 63, 64, 65]]), (read(2), torch.stack([wb[8], wa[67]])), (read(3), wa[69:70])):
        assert got.shape == want.shape and cases.error(got, want) < LIMIT[backend[1]]


def test_trace_runner_refuses_float32_where_there_are_no_such_kernels(tmp_path):
    from prism_infer_b200.models.architecture import Qwen3VLArch

    (tmp_path / "config.json").write_text(json.dumps(Qwen3VLArch.tiny().to_hf_config()))
    assert _run_trace(str(tmp_path), tmp_path, "float32", "cuda:0", []).returncode == 3


# ------------------------------------------------------------------------------- what the tests can see
def _mistakes():
    """name -> a wrong reading of one mechanism, planted in the plain statement."""

    def swapped_norms(m):
        plain = m.layer

        def layer(x, w, i, cfg):
            w = dict(w)
            p = f"l{i}."
            if p + "norm2" in w:
                w[p + "norm1"], w[p + "norm2"] = w[p + "norm2"], w[p + "norm1"]
            return plain(x, w, i, cfg)

        m.layer = layer

    def patch(name, fn):
        return lambda m: setattr(m, name, fn)

    def no_gate(y, h, w, name):
        return y

    def drop_key(q, k, v, scale):
        out = []
        for i in range(q.shape[0]):
            keep = [j for j in range(i + 1) if j != 5 or i == 5]
            s = torch.einsum("hd,jhd->hj", q[i], k[keep]) * scale
            out.append(torch.einsum("hj,jhe->he", s.softmax(-1), v[keep]))
        return torch.stack(out)

    return {
        "norm gains swapped": swapped_norms,
        "residual gate left out": patch("gated", no_gate),
        "one key lost": patch("causal_softmax_attention", drop_key),
        "step vector of the first pass in every pass": patch("loop_input", lambda x, x0, w, t: torch.cat([x, x0], -1) @ w["loop.in"].T + w["loop.step"][0]),
        "loop input in the other order": patch("loop_input", lambda x, x0, w, t: torch.cat([x0, x], -1) @ w["loop.in"].T + w["loop.step"][t]),
        "tanh gelu": patch("gelu_exact", lambda z: torch.nn.functional.gelu(z, approximate="tanh")),
        "cap left out": patch("softcap", lambda z, cap: z),
        "latent not normalised": patch("latent", lambda h, w_dkv, weight, eps: h @ w_dkv.T * weight),
    }


@pytest.mark.parametrize("name", list(_mistakes()))
def test_mistakes_would_show(model, name):
    """Each planted mistake moves the logits beyond the limits above; the other form of the activation beyond the
    32-bit limit only."""
    import importlib.util

    spec = importlib.util.spec_from_file_location("planted_oracle", os.path.join(os.path.dirname(__file__), "poralorn_oracle.py"))
    wrong = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(wrong)
    _mistakes()[name](wrong)
    cfg, arch, w, _ = model("uneven")
    toks = cases.tokens(40, arch.vocab_size, seed=8)
    e = cases.error(wrong.forward(toks, w, cfg)[0], oracle.forward(toks, w, cfg)[0])
    assert e > (4e-5 if name == "tanh gelu" else 0.06), e
