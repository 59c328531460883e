"""The Dolidra family through the engine (configuration, loading, cache rows per layer, portions, mixed batches, greedy
generation) against the plain statement in ``dolidra_oracle.py``: on the CPU in 32-bit, on a B200 in 32-bit and bf16."""

import gc
import json
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import dolidra_cases as cases  # noqa: E402
import dolidra_oracle as oracle  # noqa: E402

from prism_infer_b200 import LLM, SamplingParams  # noqa: E402
from prism_infer_b200.config import Config  # noqa: E402
from prism_infer_b200.models.architecture import DolidraArch  # noqa: E402
from prism_infer_b200.models.model_registry import family_of_config  # noqa: E402

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
CPU = ("cpu", "float32")
GPU32 = pytest.param(("cuda:0", "float32"), marks=pytest.mark.gpu, id="gpu-float32")
GPU16 = pytest.param(("cuda:0", "bfloat16"), marks=pytest.mark.gpu, id="gpu-bfloat16")
BACKENDS = [pytest.param(CPU, id="cpu"), GPU32, GPU16]
LIMIT32, LIMIT16, ROUTED16 = 5e-5, 0.05, 0.7


def check(got, want, backend, name="", where=None):
    """Every position within the limit.  In 16 bits a router may pick another expert where two logits all but tie: in models
    with routed experts nine positions of ten keep the limit and the others stay near."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    e = d.pow(2).mean(-1).sqrt() / want.double().std()
    if backend[1] == "float32":
        assert float(e.max()) < LIMIT32, (where, float(e.max()))
    elif name in cases.ROUTED:
        assert float(e.quantile(0.9)) < LIMIT16 and float(e.max()) < ROUTED16, (where, float(e.quantile(0.9)), float(e.max()))
    else:
        assert float(e.max()) < LIMIT16, (where, float(e.max()))


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


@pytest.fixture(scope="module")
def truth(model):
    """(name, length, seed) -> tokens, logits at every position, stream after every layer run."""
    made = {}

    def get(name, n, seed=0):
        if (name, n, seed) not in made:
            cfg, arch, w, _ = model(name)
            toks = cases.tokens(n, arch.vocab_size, seed=seed)
            made[name, n, seed] = (toks, *oracle.forward(toks, w, cfg))
        return made[name, n, seed]

    return get


# ---------------------------------------------------------------------------------- configuration and loading
def test_config_round_trip_and_layer_runs():
    for name, cfg in cases.CASES.items():
        arch = DolidraArch.from_hf_config(cfg)
        assert family_of_config(cfg).name == "dolidra"
        assert DolidraArch.from_hf_config(json.loads(json.dumps(arch.to_hf_config()))) == arch, name
        assert [r.layer for r in arch.layer_runs()] == oracle.layer_order(cfg)
    tiny = DolidraArch.tiny()
    assert DolidraArch.from_hf_config(tiny.to_hf_config()) == tiny


def test_config_is_checked():
    good = cases.CASES["uneven"]
    first = good["layers"][0]

    def mixer(**kw):
        return {"layers": [{**first, "mixer": {**first["mixer"], **kw}}]}

    for change in ({"layers": []}, {"loop": {"start": 2, "stop": 2, "times": 1}}, {"layers": [{**first, "type": "other"}]},
                   {"layers": [{**first, "mlp": {"kind": "x"}}]}, {"token_side": {"dim": 0}}, mixer(kv_heads=2), mixer(mask={"size": 0}),
                   mixer(rot={"base": 10.0, "dims": 26}), mixer(rot={"base": 10.0, "dims": 5}), {"layers": [{**first, "mlp": cases.moe(2, 3, 8)}]}):
        with pytest.raises(ValueError):
            DolidraArch.from_hf_config({**good, **change})
    for missing in ("vocab", "width", "norm", "token_side", "layers"):
        with pytest.raises(ValueError, match=missing):
            DolidraArch.from_hf_config({k: v for k, v in good.items() if k != missing})


def test_options_the_family_does_not_have_are_refused():
    for kw in ({"compression_mode": "scaled_fp8_kv"}, {"compression_mode": "visual_compact"}, {"tensor_parallel_size": 2}):
        with pytest.raises(ValueError):
            Config("random:dolidra-tiny", **kw)
    llm = LLM("random:dolidra-tiny", device="cpu", enforce_eager=True, kvcache_block_size=16, num_kvcache_blocks=4, max_model_len=64)
    with pytest.raises(ValueError, match="text"):
        llm.generate_images("1 2", [])


def test_loading_checks_names_and_shapes(model):
    cfg, arch, w, _ = model("uneven")
    from prism_infer_b200.models.dolidra import DolidraModel

    m = DolidraModel(arch, device="cpu", dtype=torch.float32)
    for name in ("l0.mix.lq2", "l1.mix.q.norm", "l1.mlp.e4.up", "l2.side.norm", "l0.mix.k.b"):
        with pytest.raises(KeyError, match="missing"):
            m.load((k, v) for k, v in w.items() if k != name)
    with pytest.raises(ValueError, match="side.embed"):
        m.load({**w, "side.embed": w["side.embed"][:, :-1]}.items())
    m.load({**w, "unknown.tensor": torch.zeros(3)}.items())
    assert m.weights[1].always == 2 and m.weights[1].gate_up.shape[0] == 7  # the shared width takes two blocks of the routed one


def test_environment_check_knows_the_family(model):
    from prism_infer_b200.utils.check_environment import inspect_checkpoint

    rep, errors, _ = inspect_checkpoint(model("uneven")[3], 1)
    assert rep["status"] == "pass" and not errors and rep["text"]["layer_runs"] == 5
    assert inspect_checkpoint(model("uneven")[3], 2)[1]


def test_kernel_units_exist():
    from prism_infer_b200.models.model_registry import resolve_model_family
    from prism_infer_b200.ops import build

    assert {u + ".cu" for u in resolve_model_family("dolidra").kernel_units} <= set(build._sources())


def test_cache_rows_follow_the_layer(model):
    """Every layer run has a slab of its own row width; whole pages and the first rows of a page move together in all of them."""
    from prism_infer_b200 import ops

    g = DolidraArch.from_hf_config(cases.CASES["uneven"]).kv_geometry()
    rows = (1 * (2 * 32 + 48), 2 * (48 + 32), 3 * (2 * 16 + 32))
    assert g.rows == (rows[0], rows[1], rows[2], rows[1], rows[2]) and (g.planes, g.heads, g.row) == (1, 1, max(rows))
    assert g.bytes_per_page(64, 2) == sum(g.rows) * 64 * 2
    cache = ops.KVCache(g.layers, 5, 1, 8, g.row, ops.KV_BF16, "cpu", dtype=torch.float32, planes=1, rows=g.rows)
    assert cache.bytes_per_page() == g.bytes_per_page(8, 4) and cache.payload.numel() == 5 * 8 * sum(g.rows)
    for l in range(5):
        cache.token_rows(l).copy_(torch.arange(5.)[:, None, None] * 100 + torch.arange(8.)[:, None] + l * 1000)
    ops.kv_page_copy(cache, cache, [1, 2], [3, 4], [8, 3])
    ops.kv_compact(cache, torch.tensor([8 + 7]), torch.tensor([0]))
    for l in range(5):
        t = cache.token_rows(l)
        assert t.shape == (5, 8, g.rows[l])
        assert torch.equal(t[3], t[1]) and torch.equal(t[4, :3], t[2, :3]) and float(t[4, 3, 0]) == l * 1000 + 403
        assert torch.equal(t[0, 0], t[1, 7]) and float(t[0, 1, -1]) == l * 1000 + 1


# ----------------------------------------------------------------------------------------- whole forward
@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", list(cases.CASES))
def test_whole_prompt_and_residual_stream(model, truth, name, backend):
    """Logits at every position, and the stream after every layer run."""
    cfg, arch, w, path = model(name)
    toks, want, states = truth(name, 150)
    llm = cases.engine(path, backend)
    got = cases.replay(llm, [([("a", toks)], ["a"])])["a"]
    check(got, want, backend, name)
    runner = llm.runners.runner
    from prism_infer_b200.models.common import AttnMeta

    dev, n = runner.device, len(toks)
    table = torch.arange(10, dtype=torch.int32).view(1, -1).to(dev)
    meta = AttnMeta(is_prefill=True, block_tables=table, slots=torch.arange(n).to(dev), max_q_len=n, no_history=True, total_kv=n,
                    max_kv_len=n, attended_pairs=n * n, cu_seqlens_q=torch.tensor([0, n], dtype=torch.int32).to(dev),
                    kv_lens=torch.tensor([n], dtype=torch.int32).to(dev))
    pos = torch.arange(n, dtype=torch.int32).repeat(3, 1).contiguous().to(dev)
    st = runner.model.begin_layers(torch.tensor(toks).to(dev), pos, meta, runner.kv)
    for i in range(arch.num_layer_runs):
        runner.model.advance_layers(st, 1)
        x = st.x.double().cpu()
        assert bool((x[:, arch.width:] == 0).all())
        d = (x[:, :arch.width] - states[i]).pow(2).mean(-1).sqrt() / states[i].std()
        assert float(d.max() if backend[1] == "float32" else d.quantile(0.9)) < (LIMIT32 if backend[1] == "float32" else 0.03), i
    llm.exit()


@pytest.mark.parametrize("backend", BACKENDS)
def test_first_tokens_of_a_sequence(model, backend):
    cfg, arch, w, path = model("once")
    llm = cases.engine(path, backend)
    for n in (1, 2, 3, 15, 16, 17, 18, 19):
        toks = cases.tokens(n, arch.vocab_size, seed=n)
        got = cases.replay(llm, [([("a", toks)], ["a"])])["a"]
        check(got, oracle.forward(toks, w, cfg)[0], backend, "once", n)
    llm.exit()


# ---------------------------------------------------------------------- decoding, portions, batches, pages
@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", list(cases.CASES))
def test_token_by_token_decoding_equals_the_prompt(model, truth, name, backend):
    _, _, _, path = model(name)
    toks, want, _ = truth(name, 150)
    llm = cases.engine(path, backend)
    n = 80 if name in ("once", "uneven") else 120  # from the first token, or from a prompt on
    first = [] if name in ("once", "uneven") else [([("a", toks[:30])], [])]
    got = cases.replay(llm, first + cases.portions("a", toks[30 if first else 0:n], [1]))["a"]
    check(got, want[:n], backend, name)
    llm.exit()


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name,sizes", [("ragged", [2]), ("full", [3, 37, 1]), ("once", [16]), ("uneven", [15, 17]), ("full", [64, 5]),
                                        ("ragged", [1, 2, 90]), ("wide", [2, 33]), ("many", [11])])
def test_portions_of_a_prompt(model, truth, name, sizes, backend):
    _, _, _, path = model(name)
    toks, want, _ = truth(name, 150)
    llm = cases.engine(path, backend)
    check(cases.replay(llm, cases.portions("a", toks, sizes))["a"], want, backend, name)
    llm.exit()


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", ["uneven", "full"])
def test_mixed_batches_and_reused_pages(model, truth, name, backend):
    """Portions of some requests beside single tokens of others, requests left out of steps, pages freed and used
    again by later requests; a pool that holds exactly what is live."""
    _, _, _, path = model(name)
    t = {r: truth(name, n, i) for i, (r, n) in enumerate({"a": 61, "b": 34, "c": 130, "d": 20, "e": 97}.items())}
    at = {r: 0 for r in t}

    def take(r, n):
        part = t[r][0][at[r]:at[r] + n]
        at[r] += len(part)
        return r, part

    steps = [([take("a", 30), take("b", 2)], []), ([take("a", 1), take("b", 15), take("c", 64)], []), ([take("c", 2), take("a", 1)], []),
             ([take("a", 1), take("b", 1), take("c", 1)], []), ([take("b", 16), take("a", 1)], ["b"]),
             ([take("d", 20), take("c", 33), take("a", 1)], ["d"]), ([take("e", 80), take("a", 26), take("c", 1)], ["a"])]
    while at["c"] < 130 or at["e"] < 97:
        entries = [take(r, n) for r, n in (("c", 1), ("e", 1)) if at[r] < len(t[r][0])]
        steps.append((entries, [r for r, _ in entries if at[r] == len(t[r][0])]))
    llm = cases.engine(path, backend, num_kvcache_blocks=17)
    free = llm.scheduler.block_manager.gpu.num_free
    for repeat in range(2):  # the second time over other pages, with the first run's keys still in them
        got = cases.replay(llm, steps)
        for r in t:
            check(got[r], t[r][1], backend, name, (r, repeat))
        assert llm.scheduler.block_manager.gpu.num_free == free
    llm.exit()


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("page", [32, 64, 256])
def test_page_sizes(model, truth, page, backend):
    """Pages smaller than, as large as and larger than a key tile."""
    _, _, _, path = model("once")
    toks, want, _ = truth("once", 150)
    llm = cases.engine(path, backend, kvcache_block_size=page, num_kvcache_blocks=-(-640 // page))
    check(cases.replay(llm, cases.portions("a", toks, [70, 2, 33, 1, 1, 9]))["a"], want, backend, "once")
    llm.exit()


@pytest.mark.parametrize("backend", BACKENDS)
def test_long_decoding(model, truth, backend):
    """Windows, kept tokens and key tiles pass over a long run of decoded tokens."""
    _, _, _, path = model("once")
    toks, want, _ = truth("once", 400, 11)
    llm = cases.engine(path, backend)
    got = cases.replay(llm, [([("a", toks[:9])], [])] + cases.portions("a", toks[9:], [1]))["a"]
    check(got, want, backend, "once")
    llm.exit()


@pytest.mark.gpu
def test_long_prompts_take_the_grouped_and_persistent_kernels(cuda_device, model):
    """More tokens in a step than the small-token forms take: row GEMM epilogues and gathered expert tiles."""
    cfg, arch, w, path = model("uneven")
    toks = {r: cases.tokens(n, arch.vocab_size, seed=n) for r, n in (("a", 390), ("b", 270))}
    for backend in (("cuda:0", "float32"), ("cuda:0", "bfloat16")):
        llm = cases.engine(path, backend)
        llm2 = cases.replay(llm, [([(r, t) for r, t in toks.items()], list(toks))])
        for r, t in toks.items():
            check(llm2[r], oracle.forward(t, w, cfg)[0], backend, "uneven", r)
        llm.check_device_status()
        llm.exit()


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
    name = "uneven" if backend[1] == "float32" else "once"  # routed experts only where no logits all but tie
    cfg, arch, w, path = model(name)
    shared = cases.tokens(48, arch.vocab_size, seed=30)
    prompts = [shared + cases.tokens(n, arch.vocab_size, seed=40 + n) for n in (1, 9, 30)] + [cases.tokens(5, arch.vocab_size, seed=50)]
    llm = cases.engine(path, backend, **options)
    sp = SamplingParams(temperature=0.0, max_tokens=20, ignore_eos=False)
    out = llm.generate(prompts, sp, use_tqdm=False)
    if options.get("enable_prefix_caching"):
        out = llm.generate(prompts, sp, use_tqdm=False)  # pages of the first round are hit
    for p, o in zip(prompts, out):
        assert len(o["token_ids"]) == 20
        _greedy_ok(o["token_ids"], p, w, cfg, 1e-3 if backend[1] == "float32" else 0.4)
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
    llm = LLM("random:dolidra-8b-like-4layer" if dtype == "auto" else "random:dolidra-tiny", dtype=dtype, gpu_memory_utilization=0.3,
              max_num_seqs=8, max_num_batched_tokens=2048, cpu_kv_cache_ratio=0.0)
    sizing = llm.graph_metadata()["kv_sizing"]
    assert sizing["budget_bytes"] > 0 and llm.scheduler.block_manager.gpu.num_blocks > 100
    prompts = [cases.tokens(n, 200, seed=n) for n in (1700, 3, 41)]
    together = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True), use_tqdm=False)
    assert all(len(o["token_ids"]) == 6 for o in together)
    llm.check_device_status()
    llm.exit()
    del llm
    gc.collect()  # the cache takes a third of the device: give it back before the next test
    torch.cuda.empty_cache()


@pytest.mark.parametrize("backend", BACKENDS)
def test_served_over_http(model, backend):
    """The serving runtime answers text requests with the same greedy tokens."""
    import asyncio

    import httpx

    from prism_infer_b200.serving.app import create_app
    from prism_infer_b200.serving.runtime import ServingRuntime

    cfg, arch, w, path = model("once")
    prompt = cases.tokens(10, arch.vocab_size, seed=6)
    runtime = ServingRuntime(lambda: cases.engine(path, backend))
    runtime.start()
    app = create_app(runtime, model_name="dolidra", manage_runtime=False)

    async def scenario():
        async with httpx.AsyncClient(transport=httpx.ASGITransport(app=app), base_url="http://t", timeout=60.0) as client:
            r = await client.post("/v1/generate", json={"prompt": " ".join(map(str, prompt)), "sampling": {"max_tokens": 6, "ignore_eos": True}})
            assert r.status_code == 200, r.text
            _greedy_ok(r.json()["token_ids"], prompt, w, cfg, 1e-3 if backend[1] == "float32" else 0.4)

    try:
        asyncio.run(scenario())
    finally:
        runtime.stop()


# ----------------------------------------------------------------------------------------- trace runner
@pytest.mark.parametrize("backend", BACKENDS)
def test_trace_runner(model, truth, tmp_path, backend):
    _, arch, _, path = model("once")
    (a, wa, _), (b, wb, _) = truth("once", 70, 1), truth("once", 9, 2)
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": a[:66], "want": [0, 63, 64, 65]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[:8], "want": []}, {"id": "a", "tokens": a[66:67], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[8:], "want": [0]}, {"id": "a", "tokens": a[67:68], "want": [0]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": a[68:], "want": [1]}], "end": ["a"]}]
    cmd = [os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", backend[1], "--out", str(tmp_path), "--max-tokens", "256",
           "--device", backend[0]]
    res = subprocess.run(cmd, input="".join(json.dumps(x) + "\n" for x in lines), capture_output=True, text=True, timeout=240)
    assert res.returncode == 0, res.stderr
    assert [x for x in res.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    assert not (tmp_path / "1.f32").exists()

    def read(step):
        return torch.frombuffer(bytearray((tmp_path / f"{step}.f32").read_bytes()), dtype=torch.float32).view(-1, arch.vocab_size)

    for got, want in ((read(0), wa[[0, 63, 64, 65]]), (read(2), torch.stack([wb[8], wa[67]])), (read(3), wa[69:70])):
        assert got.shape == want.shape
        check(got, want, backend, "once")


# ------------------------------------------------------------------------------- what the tests can see
def _mistakes():
    """name -> a wrong reading of one mechanism, planted in the plain statement."""

    def patch(attr, fn):
        return lambda m: setattr(m, attr, fn)

    def window(shift, keep_shift=0):
        return patch("visible", lambda i, size, keep=0: [j for j in range(i + 1) if i - j < size + shift or j < max(0, keep + keep_shift)])

    def unscaled(m):
        plain = m.frequencies
        m.frequencies = lambda rot: plain({k: v for k, v in rot.items() if k != "scaling"})

    def interleaved(m):
        def rotate(x, rot, first=0):
            d = rot["dims"]
            a = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * m.frequencies(rot)
            c, s = a.cos()[:, None], a.sin()[:, None]
            u, v = x[..., 0:d:2], x[..., 1:d:2]
            return torch.cat([torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2), x[..., d:]], -1)

        m.rotate = rotate

    def per_head_norm(m):
        plain = m.norm

        def norm(x, weight, eps):
            if x.shape[-1] in (160, 80):  # the whole query and key rows of the routed layer
                return plain(x.view(x.shape[0], -1, 40), weight.view(-1, 40), eps).flatten(1)
            return plain(x, weight, eps)

        m.norm = norm

    def all_experts_softmax(m):
        plain = m.route

        def route(h, w_router, top):
            z = torch.softmax(h @ w_router.T, -1)
            return [[(e, float(z[t, e])) for e, _ in chosen] for t, chosen in enumerate(plain(h, w_router, top))]

        m.route = route

    return {
        "window one longer": window(1), "window one shorter": window(-1), "one kept token less": window(0, -1), "one kept token more": window(0, 1),
        "second map left out": patch("difference_weight", lambda w, p, diff: 0.0),
        "constant left out of the map weight": patch("combine_maps", lambda a1, a2, lam, diff, eps: oracle.rms(a1 - (lam - diff) * a2, eps) * (1 - diff)),
        "difference not normalised": patch("combine_maps", lambda a1, a2, lam, diff, eps: (a1 - lam * a2) * (1 - diff)),
        "frequencies not scaled": unscaled, "neighbouring pairs rotated": interleaved,
        "query and key norm per head": per_head_norm, "head gate left out": patch("sigmoid", lambda z: torch.ones_like(z)),
        "softmax over all experts": all_experts_softmax,
        "side table left out": patch("token_side", lambda x, tokens, w, i, cfg: 0.0 * x),
        "side part of another layer": lambda m: setattr(m, "token_side", (lambda plain: lambda x, tokens, w, i, cfg: plain(
            x, tokens, {**w, "side.embed": w["side.embed"].roll(cfg["token_side"]["dim"], 1)}, i, cfg))(m.token_side)),
        "exact gelu": patch("gelu_tanh", lambda z: 0.5 * z * (1.0 + torch.erf(z / 2.0 ** 0.5))),
    }


@pytest.mark.parametrize("name", list(_mistakes()))
def test_mistakes_would_show(model, name):
    """Each planted mistake moves the logits beyond the limits above; the other form of the activation beyond the
    32-bit limit only."""
    import importlib.util

    spec = importlib.util.spec_from_file_location("planted_oracle", os.path.join(os.path.dirname(__file__), "dolidra_oracle.py"))
    wrong = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(wrong)
    _mistakes()[name](wrong)
    cfg, arch, w, _ = model("uneven")
    toks = cases.tokens(50, arch.vocab_size, seed=8)
    e = cases.error(wrong.forward(toks, w, cfg)[0], oracle.forward(toks, w, cfg)[0])
    assert e > (1e-4 if name == "exact gelu" else 0.06), e
