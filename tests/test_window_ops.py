"""Windowed attention: preparation of queries and cache rows, masks, maps, gates and splits, each against the plain float64
statement.  CPU statements, and the kernels on a B200 (bf16 also through the kernel that serves any head width)."""

import dataclasses
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import dolidra_oracle as oracle  # noqa: E402
from op_helpers import BACKENDS, GPU16, close, rand  # noqa: E402

from prism_infer_b200 import ops  # noqa: E402
from prism_infer_b200.models.architecture import RotaryArch  # noqa: E402
from prism_infer_b200.ops import window  # noqa: E402
from prism_infer_b200.ops.latent import Branch  # noqa: E402


def spec(heads, kv_heads, dim, vdim, win, keep=0, maps=1, rot=0, gate=False, lam=0.0, gain=1.0, scale=None, eps=1e-5):
    return window.WindowSpec(heads=heads, kv_heads=kv_heads, maps=maps, dim=dim, vdim=vdim, rot_dims=rot, window=win, keep_first=keep,
                             gate=gate, lam=lam, gain=gain, scale=dim ** -0.5 if scale is None else scale, eps=eps)


SPECS = {
    "plain": spec(4, 2, 64, 64, 40, 6, gate=True),
    "pair-of-maps": spec(4, 1, 32, 64, 50, maps=2, lam=0.7, gain=0.4),
    "odd-group": spec(6, 2, 48, 80, 33, 1, gate=True),
    "own-keys": spec(3, 3, 16, 96, 100, 130),
    "negative-weight": spec(5, 5, 112, 128, 64, maps=2, lam=-1.6, gain=0.25),
    "ragged": spec(6, 3, 13, 21, 17, 3, maps=2, lam=1.1, gain=0.6),
    "widest": spec(8, 2, 128, 128, 129, 64, gate=True),
    "widest-maps": spec(2, 1, 128, 128, 63, maps=2, lam=0.9, gain=0.1),
    "two-row-tiles": spec(24, 1, 32, 48, 70, 2),
    "many-rows": spec(40, 2, 16, 32, 35, maps=2, lam=0.5, gain=0.5),
    "wide": spec(2, 1, 160, 200, 30, 4, gate=True),
    "wider": spec(2, 1, 272, 264, 30, 4, gate=True),
    "alone": spec(4, 2, 32, 32, 1),
    "everything": spec(4, 2, 32, 32, 100000),
}


# -------------------------------------------------------------------------------------------- frequencies
@pytest.mark.parametrize("rot", [
    {"base": 5000.0, "dims": 14}, {"base": 100.0, "dims": 2},
    {"base": 20000.0, "dims": 40, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 300}},
    {"base": 9.0, "dims": 6, "scaling": {"factor": 3.0, "low": 2.0, "high": 2.5, "original": 40}}])
def test_frequencies(rot):
    s = rot.get("scaling")
    arch = RotaryArch(rot["base"], rot["dims"], *((s["factor"], s["low"], s["high"], s["original"]) if s else ()))
    got, want = torch.tensor(arch.inv_freq(), dtype=torch.float64), oracle.frequencies(rot)
    assert torch.allclose(got, want, rtol=1e-12)
    if s and rot["dims"] == 40:  # all three bands are there
        plain = oracle.frequencies({k: v for k, v in rot.items() if k != "scaling"})
        ratio = want / plain
        assert bool((ratio == 1).any()) and bool((ratio < 1 / 7.9).any()) and bool(((ratio > 0.13) & (ratio < 0.99)).any())


# --------------------------------------------------------------------------------------------- preparation
def pad_heads(t, heads, real, padded):
    """[..., heads * real] -> [..., heads * padded]"""
    t = t.view(*t.shape[:-1], heads, real)
    return torch.nn.functional.pad(t, (0, padded - real)).flatten(-2)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("source", ["slabs", "rows"])
@pytest.mark.parametrize("T", [5, 60, 300])
@pytest.mark.parametrize("name,bias,norm,rot", [("pair-of-maps", True, False, 24), ("plain", False, True, 16), ("ragged", True, True, 12),
                                                ("own-keys", False, False, 0), ("widest", True, True, 128), ("odd-group", False, True, 2)])
def test_prepare(backend, source, name, bias, norm, rot, T):
    device, dtype = backend
    sp = dataclasses.replace(SPECS[name], rot_dims=rot)
    page, H, G, M, d, e = 16, sp.heads, sp.kv_heads, sp.maps, sp.dim, sp.vdim
    freq = torch.tensor(oracle.frequencies({"base": 300.0, "dims": rot}).tolist())
    parts = [(H * M, d, sp.dq), (G * M, d, sp.dq), (G, e, sp.dv)]

    def stack(seed, rows=T):
        real = [rand(rows, n * r, seed=seed + i) for i, (n, r, _) in enumerate(parts)]
        real.append(rand(rows, H, seed=seed + 3))
        flat = torch.cat([pad_heads(x, n, r, p) for x, (n, r, p) in zip(real, parts)] + ([real[3]] if sp.gate else []), 1)
        return real, torch.nn.functional.pad(flat, (0, sp.proj_cols - flat.shape[1]))

    (q, k, v, zg), flat = stack(1)
    (bq, bk, bv, bg), flat_b = stack(20, 1)
    qn, kn = 0.5 + rand(H * M * d, seed=40).abs(), 0.5 + rand(G * M * d, seed=41).abs()
    w = window.WindowWeights(
        bias=flat_b[0].to(device, dtype) if bias else None,
        q_norm=pad_heads(qn, H * M, d, sp.dq).to(device, dtype) if norm else None,
        k_norm=pad_heads(kn, G * M, d, sp.dq).to(device, dtype) if norm else None, inv_freq=freq.float().to(device))
    if source == "slabs":  # three slabs that add up
        a, b = rand(T, sp.proj_cols, seed=50), rand(T, sp.proj_cols, seed=51)
        proj = Branch(slabs=torch.stack([a, b, flat - a - b]).to(device))
    else:
        proj = Branch(rows=flat.to(device, dtype))
    g = torch.Generator().manual_seed(T)
    positions = torch.cat([torch.tensor([0, 3, 17, 400, 2]), torch.randint(0, 500, (T - 5,), generator=g)]).int()
    slots = torch.randperm(16 * page * 2, generator=g)[:T]
    slots[2] = -1
    cache = ops.KVCache(2, 32, 1, page, sp.k_cols + sp.v_cols, ops.KV_BF16, device, dtype=dtype, planes=1)
    cache.payload.fill_(7.0)
    q_got, gate = window.qkv_prepare(proj, sp, w, positions.to(device), slots.to(device), cache, 1)

    def expected(x, b, weight, heads):
        x = x.double() + (b.double() if bias else 0.0)
        if norm:
            x = oracle.norm(x, weight.double(), sp.eps)
        x = x.view(T, heads, d)
        return torch.cat([oracle.rotate(x[t:t + 1], {"base": 300.0, "dims": rot}, first=int(positions[t])) for t in range(T)])

    wq, wk = expected(q, bq, qn, H * M), expected(k, bk, kn, G * M)
    close(q_got, torch.nn.functional.pad(wq, (0, sp.dq - d)).flatten(1), dtype, tol32=1e-4)
    wv = v.double() + (bv.double() if bias else 0.0)
    row = torch.cat([torch.nn.functional.pad(wk, (0, sp.dq - d)).flatten(1), pad_heads(wv, G, e, sp.dv)], 1)
    flat_cache = cache.token_rows(1).reshape(-1, row.shape[1])
    keep = slots >= 0
    close(flat_cache[slots[keep].to(device)], row[keep], dtype, tol32=1e-4)
    untouched = torch.ones(32 * page, dtype=torch.bool)
    untouched[slots[keep]] = False
    assert bool((flat_cache.cpu()[untouched] == 7.0).all()) and bool((cache.token_rows(0) == 7.0).all())
    assert (gate is not None) == sp.gate
    if sp.gate:
        close(gate, oracle.sigmoid(zg.double() + (bg.double() if bias else 0.0)), torch.float32)


# ----------------------------------------------------------------------------------------------- attention
def paged(sp, seqs, device, dtype, page, seed=0, noise=1.0):
    """Random keys, values and queries of sequences ``(kv_len, q_len)`` and the cache that holds them in shuffled pages, the free
    pages and the rest of the last page filled with large junk."""
    H, G, M = sp.heads, sp.kv_heads, sp.maps
    per = [-(-n // page) for n, _ in seqs]
    blocks = sum(per) + 2
    order = torch.randperm(blocks, generator=torch.Generator().manual_seed(seed + 99)).tolist()
    tables = torch.full((len(seqs), max(per) + 1), -1, dtype=torch.int32)
    data = []
    rows = torch.full((blocks, page, sp.k_cols + sp.v_cols), 50.0)
    for s, (n, ql) in enumerate(seqs):
        q = rand(ql, H, M, sp.dim, seed=seed + 10 * s, scale=noise)
        k = rand(n, G, M, sp.dim, seed=seed + 10 * s + 1, scale=noise)
        v = rand(n, G, sp.vdim, seed=seed + 10 * s + 2)
        data.append([q, k, v])
        for b in range(per[s]):
            tables[s, b] = order.pop()
    return data, tables, rows


def fill(sp, data, tables, rows, device, dtype, page):
    pad = torch.nn.functional.pad
    for s, (_, k, v) in enumerate(data):
        n = k.shape[0]
        flat = torch.cat([pad(k, (0, sp.dq - sp.dim)).flatten(1), pad(v, (0, sp.dv - sp.vdim)).flatten(1)], 1)
        pos = torch.arange(n)
        rows[tables[s, pos // page].long(), pos % page] = flat
    cache = ops.KVCache(1, rows.shape[0], 1, page, rows.shape[2], ops.KV_BF16, device, dtype=dtype, planes=1)
    cache.token_rows(0).copy_(rows)
    q = torch.cat([pad(x[0], (0, sp.dq - sp.dim)).flatten(1) for x in data])
    return cache, q.to(device, dtype).contiguous()


def want_attention(sp, data, gate):
    out, at = [], 0
    for q, k, v in data:
        n, ql = k.shape[0], q.shape[0]
        maps = [oracle.masked_attention(q[:, :, m].double(), k[:, :, m].double(), v.double(), sp.scale, sp.window, sp.keep_first,
                                        first=n - ql) for m in range(sp.maps)]
        o = maps[0] if sp.maps == 1 else oracle.rms(maps[0] - sp.lam * maps[1], sp.eps) * sp.gain
        if gate is not None:
            o = o * gate[at:at + ql, :, None].double()
        at += ql
        out.append(torch.nn.functional.pad(o, (0, sp.dv - sp.vdim)).flatten(1))
    return torch.cat(out)


def run(sp, data, tables, rows, backend, page, *, decode, nsplit=0, simple=False):
    device, dtype = backend
    cache, q = fill(sp, data, tables, rows, device, dtype, page)
    gate = torch.sigmoid(rand(q.shape[0], sp.heads, seed=77)) if sp.gate else None
    lens = torch.tensor([k.shape[0] for _, k, _ in data], dtype=torch.int32)
    kw = {}
    if not decode:
        cu = torch.tensor([0] + [x[0].shape[0] for x in data]).cumsum(0).to(torch.int32)
        kw = dict(cu_seqlens_q=cu.to(device), max_q_len=max(x[0].shape[0] for x in data))
    got = window.window_attention(q, sp, gate.to(device) if gate is not None else None, cache, 0, tables.to(device), lens.to(device),
                                  nsplit=nsplit, simple=simple, **kw)
    if device != "cpu":
        from prism_infer_b200.ops import native

        native.check_status()
    return got, want_attention(sp, data, gate)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", list(SPECS))
def test_prompts_and_portions(backend, name):
    """Whole prompts, portions behind a history down to two tokens, single tokens between them; one batch, shuffled pages."""
    sp = SPECS[name]
    seqs = [(150, 150), (1, 1), (201, 2), (70, 33), (130, 1), (300, 140), (64, 64)]
    data, tables, rows = paged(sp, seqs, *backend, 16)
    got, want = run(sp, data, tables, rows, backend, 16, decode=False)
    close(got, want, backend[1], tol16=0.02)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", list(SPECS))
def test_decode(backend, name):
    sp = SPECS[name]
    seqs = [(n, 1) for n in (1, 2, 40, 41, 63, 64, 65, 128, 200, 333, 17)]
    for nsplit in ([0] if backend[0] == "cpu" else [0, 1, 2, 5, 32]):
        data, tables, rows = paged(sp, seqs, *backend, 64)
        got, want = run(sp, data, tables, rows, backend, 64, decode=True, nsplit=nsplit)
        close(got, want, backend[1], tol16=0.02)


@pytest.mark.parametrize("backend", [GPU16])
@pytest.mark.parametrize("name", ["plain", "pair-of-maps", "ragged"])
def test_kernel_for_any_width_in_16_bits(backend, name):
    sp = SPECS[name]
    for decode, seqs in ((False, [(90, 90), (120, 2)]), (True, [(33, 1), (150, 1)])):
        data, tables, rows = paged(sp, seqs, *backend, 16)
        got, want = run(sp, data, tables, rows, backend, 16, decode=decode, simple=True)
        close(got, want, backend[1], tol16=0.02)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("maps", [1, 2])
@pytest.mark.parametrize("win,keep", [(40, 6), (64, 0), (65, 64), (128, 70), (17, 1), (1, 2), (200, 3)])
def test_edges_of_the_window_and_of_the_kept_tokens(backend, decode, maps, win, keep):
    """One key that outscores all others by far, placed just inside and just outside each edge: the output is that key's value, or
    does not know it.  Positions around tile and page borders."""
    sp = spec(4, 2, 32, 48, win, keep, maps=maps, lam=0.5, gain=1.0, scale=0.3)
    for i in (250, 255, 256, 257, 191):
        # the newest key outside the window, the oldest inside, kept and first not kept, itself; those that exist
        for j in {i - win, i - win + 1, keep - 1, keep, 0, i, 64, 63} & set(range(i + 1)):
            data, tables, rows = paged(sp, [(i + 1, 1 if decode else 20)], *backend, 64, seed=i, noise=0.3)
            q, k, v = data[0]
            q[-1] = q[-1, :1]                                   # one direction for all heads of the query
            for m in range(maps):
                d = q[-1, 0, m] / q[-1, 0, m].norm()
                q[-1, :, m] = (4.0 * d).to(torch.bfloat16).float()
                k[j, :, m] = (40.0 * d).to(torch.bfloat16).float()
            v[j] = v[j] + 3.0
            got, want = run(sp, data, tables, rows, backend, 64, decode=decode)
            close(got[-1:], want[-1:], backend[1], tol16=0.02, tol32=1e-4)
            seen = j in oracle.visible(i, win, keep)
            if maps == 1:
                head = v[j].repeat_interleave(2, 0).double()
                assert (float((want[-1].view(4, 48) - head).abs().max()) < 0.05) == seen


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("decode", [False, True])
def test_rising_scores(backend, decode):
    """Scores that grow by hundreds along the keys: the running maximum is raised again and again."""
    for maps in (1, 2):
        sp = spec(2, 1, 16, 32, 400, maps=maps, lam=0.3, gain=1.0, scale=1.0)
        data, tables, rows = paged(sp, [(300, 1 if decode else 200)], *backend, 64, noise=0.1)
        q, k, _ = data[0]
        q[..., 0] = 8.0
        k[..., 0] = (torch.arange(300.0) * 0.25).view(-1, 1, 1).to(torch.bfloat16).float()
        got, want = run(sp, data, tables, rows, backend, 64, decode=decode)
        close(got, want, backend[1], tol16=0.02, tol32=5e-4)


@pytest.mark.parametrize("backend", BACKENDS)
def test_padding_rows_of_a_decode_step(backend):
    """A row without context (padding of a captured batch) gives zeros and disturbs nothing."""
    sp = SPECS["pair-of-maps"]
    data, tables, rows = paged(sp, [(50, 1), (90, 1)], *backend, 16)
    device, dtype = backend
    cache, q = fill(sp, data, tables, rows, device, dtype, 16)
    q = torch.cat([q[:1], q[:1], q[1:]])
    bt = torch.cat([tables[:1], torch.full_like(tables[:1], -1), tables[1:]])
    got = window.window_attention(q, sp, None, cache, 0, bt.to(device), torch.tensor([50, 0, 90], dtype=torch.int32).to(device))
    want = want_attention(sp, data, None)
    close(got[[0, 2]], want, dtype, tol16=0.02)
    assert bool((got[1] == 0).all())


# ---------------------------------------------------------------------------------------------- side table
@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("source", ["slabs", "rows"])
def test_token_side_gate(backend, source):
    device, dtype = backend
    T, V, L, D = 37, 19, 3, 48
    z, table = rand(T, D, seed=1, scale=2.0), rand(V, L, D, seed=2)
    ids = torch.randint(0, V, (T,), generator=torch.Generator().manual_seed(3))
    a = rand(T, D, seed=4)
    b = Branch(slabs=torch.stack([a, z - a]).to(device)) if source == "slabs" else Branch(rows=z.to(device, dtype))
    got = window.token_side_gate(b, table.to(device, dtype), 2, ids.to(device))
    close(got, oracle.gelu_tanh(z.double()) * table[ids, 2].double(), dtype)
