"""Attention with bounded scores, sinks, norms per head, values that are the keys and keys of another layer; scored routing with
groups, identity experts and a gated shared expert; the stream update's offset norms.  Each against the plain float64 statement:
CPU statements, and the kernels on a B200."""

import dataclasses
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import bokorax_oracle as oracle  # noqa: E402
from op_helpers import BACKENDS, GPU16, close, rand  # noqa: E402
from test_window_ops import fill, pad_heads, paged  # noqa: E402

from prism_infer_b200 import ops  # noqa: E402
from prism_infer_b200.models.architecture import NO_WINDOW, RotaryArch  # noqa: E402
from prism_infer_b200.ops import latent as lat  # noqa: E402
from prism_infer_b200.ops import moe, window  # noqa: E402
from prism_infer_b200.ops.latent import Branch  # noqa: E402


def spec(heads, kv_heads, dim, vdim, win=NO_WINDOW, *, cap=0.0, rot=0, gate=False, tied=False, shared=False, head_norm=True, scale=None):
    return window.WindowSpec(heads=heads, kv_heads=kv_heads, maps=1, dim=dim, vdim=vdim, rot_dims=rot, window=win, keep_first=0, gate=gate,
                             scale=1.5 * dim ** -0.5 if scale is None else scale, eps=3e-4, head_norm=head_norm, tied=tied, shared=shared,
                             softcap=cap)


def status(device):
    if device != "cpu":
        from prism_infer_b200.ops import native

        native.check_status()


def test_frequencies_all_divided():
    for rot in ({"base": 700.0, "dims": 10, "scaling": {"factor": 2.5}}, {"base": 50.0, "dims": 2}):
        arch = RotaryArch(rot["base"], rot["dims"], (rot.get("scaling") or {"factor": 0.0})["factor"])
        assert torch.allclose(torch.tensor(arch.inv_freq(), dtype=torch.float64), oracle.frequencies(rot), rtol=1e-12)


# --------------------------------------------------------------------------------------------- preparation
PREPARE = {
    # norms per head: units of a head in a quarter of a warp up to a whole one, more than a warp, and widths that go element by element
    "small": spec(6, 2, 32, 48, rot=32, gate=True), "partial": spec(4, 2, 40, 24, rot=16, gate=True), "ragged": spec(3, 3, 13, 7, rot=6),
    "wide": spec(2, 1, 128, 128, rot=128, gate=True), "mostly-unrotated": spec(4, 1, 128, 64, rot=16), "wider": spec(2, 2, 256, 32, rot=24),
    "odd-half": spec(5, 1, 48, 16, rot=20, gate=True), "no-rotation": spec(2, 1, 64, 64), "many": spec(40, 8, 64, 64, rot=64),
    # values that are the keys, norm over whole rows; queries alone
    "tied": spec(4, 2, 48, 48, rot=32, tied=True, head_norm=False), "tied-ragged": spec(3, 3, 19, 19, rot=14, tied=True, head_norm=False),
    "tied-many": spec(24, 24, 96, 96, rot=96, tied=True, head_norm=False), "tied-per-head": spec(4, 2, 32, 32, rot=16, tied=True, gate=True),
    "shared": spec(6, 2, 32, 48, rot=32, gate=True, shared=True), "shared-ragged": spec(3, 1, 13, 7, rot=6, shared=True),
    "shared-whole": spec(4, 2, 48, 32, rot=24, shared=True, head_norm=False),
}


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("source", ["slabs", "rows"])
@pytest.mark.parametrize("T", [4, 70, 300])
@pytest.mark.parametrize("name", list(PREPARE))
def test_prepare(backend, source, T, name):
    device, dtype = backend
    sp = PREPARE[name]
    H, G, d, e, page = sp.heads, sp.kv_heads, sp.dim, sp.vdim, 16
    rot = {"base": 300.0, "dims": sp.rot_dims}
    q, k, v, z = rand(T, H * d, seed=1), rand(T, G * d, seed=2), rand(T, G * e, seed=3), rand(T, H, seed=4)
    parts = [pad_heads(q, H, d, sp.dq)]
    if not sp.shared:
        parts += [pad_heads(k, G, d, sp.dq)] + ([] if sp.tied else [pad_heads(v, G, e, sp.dv)])
    flat = torch.cat(parts + ([z] if sp.gate else []), 1)
    assert sp.gate_row == sum(p.shape[1] for p in parts)
    flat = torch.nn.functional.pad(flat, (0, sp.proj_cols - flat.shape[1]))
    if source == "slabs":
        a = rand(T, sp.proj_cols, seed=50)
        proj = Branch(slabs=torch.stack([a, flat - a]).to(device))
    else:
        proj = Branch(rows=flat.to(device, dtype))
    qn, kn = (0.5 + rand((d if sp.head_norm else n * d), seed=s).abs() for n, s in ((H, 40), (G, 41)))

    def packed(weight, heads):
        return (pad_heads(weight, 1 if sp.head_norm else heads, d, sp.dq)).to(device, dtype)

    w = window.WindowWeights(q_norm=packed(qn, H), k_norm=None if sp.shared else packed(kn, G), inv_freq=oracle.frequencies(rot).float().to(device))
    g = torch.Generator().manual_seed(T)
    positions, slots = torch.randint(0, 400, (T,), generator=g).int(), torch.randperm(32 * page, generator=g)[:T]
    slots[2] = -1
    cache = ops.KVCache(1, 32, 1, page, sp.k_cols + sp.v_cols, ops.KV_BF16, device, dtype=dtype, planes=1)
    cache.payload.fill_(7.0)
    q_got, gate = window.qkv_prepare(proj, sp, w, positions.to(device), slots.to(device), cache, 0)
    status(device)

    def expected(x, weight, heads):
        x, weight = x.double(), weight.double()
        x = oracle.rms(x.view(T, heads, d), sp.eps) * weight if sp.head_norm else (oracle.rms(x, sp.eps) * weight).view(T, heads, d)
        return torch.cat([oracle.rotate(x[t:t + 1], rot, first=int(positions[t])) for t in range(T)])

    close(q_got, torch.nn.functional.pad(expected(q, qn, H), (0, sp.dq - d)).flatten(1), dtype, tol32=1e-4)
    rows = cache.token_rows(0).reshape(32 * page, -1)
    keep = slots >= 0
    untouched = torch.ones(32 * page, dtype=torch.bool)
    if sp.shared:
        assert bool((rows == 7.0).all())
    else:
        values = pad_heads(k, G, d, sp.dq) if sp.tied else pad_heads(v, G, e, sp.dv)
        want = torch.cat([torch.nn.functional.pad(expected(k, kn, G), (0, sp.dq - d)).flatten(1), values.double()], 1)
        close(rows[slots[keep].to(device)], want[keep], dtype, tol32=1e-4)
        untouched[slots[keep]] = False
        assert bool((rows.cpu()[untouched] == 7.0).all())
    assert (gate is not None) == sp.gate
    if sp.gate:
        close(gate, oracle.sigmoid(z.double()), torch.float32)


# ----------------------------------------------------------------------------------------------- attention
ATTEND = {
    "all": (spec(6, 2, 64, 48, cap=5.0, gate=True), True), "cap": (spec(4, 2, 32, 32, cap=2.0), False), "sink": (spec(4, 4, 48, 16), True),
    "window": (spec(4, 2, 128, 128, 40, cap=8.0), True), "many-rows": (spec(24, 1, 32, 48, cap=3.0, gate=True), True),
    "odd-group": (spec(5, 1, 112, 96, cap=30.0), True), "ragged": (spec(6, 3, 13, 21, 17, cap=1.0), True), "wide": (spec(2, 1, 160, 200, cap=4.0, gate=True), True),
    "wider": (spec(2, 1, 272, 264, cap=4.0), True), "plain": (spec(4, 2, 64, 64), False),
}


def sinks(n, top=3.0):
    """From far below the scores to far above them."""
    return torch.linspace(-12.0, top, n).to(torch.bfloat16).float()


def run(sp, data, tables, rows, backend, page, *, decode, nsplit=0, simple=False, sink=None):
    device, dtype = backend
    cache, q = fill(sp, data, tables, rows, device, dtype, page)
    gate = torch.sigmoid(rand(q.shape[0], sp.heads, seed=77)) if sp.gate else None
    lens = torch.tensor([k.shape[0] for _, k, _ in data], dtype=torch.int32)
    kw = {}
    if not decode:
        cu = torch.tensor([0] + [x[0].shape[0] for x in data]).cumsum(0).to(torch.int32)
        kw = dict(cu_seqlens_q=cu.to(device), max_q_len=max(x[0].shape[0] for x in data))
    got = window.window_attention(q, sp, gate.to(device) if gate is not None else None, cache, 0, tables.to(device), lens.to(device),
                                  nsplit=nsplit, simple=simple, sink=None if sink is None else sink.to(device), **kw)
    status(device)
    out, at = [], 0
    for q, k, v in data:
        ql = q.shape[0]
        o = oracle.attend(q[:, :, 0].double(), k[:, :, 0].double(), v.double(), sp.scale, window=sp.window, cap=sp.softcap,
                          sink=None if sink is None else sink.double(), first=k.shape[0] - ql)
        if gate is not None:
            o = o * gate[at:at + ql, :, None].double()
        at += ql
        out.append(torch.nn.functional.pad(o, (0, sp.dv - sp.vdim)).flatten(1))
    return got, torch.cat(out)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", list(ATTEND))
def test_prompts_and_portions(backend, name):
    sp, has_sink = ATTEND[name]
    seqs = [(150, 150), (1, 1), (201, 2), (70, 33), (130, 1), (300, 140), (64, 64)]
    data, tables, rows = paged(sp, seqs, *backend, 16)
    got, want = run(sp, data, tables, rows, backend, 16, decode=False, sink=sinks(sp.heads) if has_sink else None)
    close(got, want, backend[1], tol16=0.02)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", list(ATTEND))
def test_decode(backend, name):
    sp, has_sink = ATTEND[name]
    seqs = [(n, 1) for n in (1, 2, 40, 41, 63, 64, 65, 128, 200, 333, 17)]
    for nsplit in ([0] if backend[0] == "cpu" else [0, 1, 2, 5, 32]):
        data, tables, rows = paged(sp, seqs, *backend, 64)
        got, want = run(sp, data, tables, rows, backend, 64, decode=True, nsplit=nsplit, sink=sinks(sp.heads) if has_sink else None)
        close(got, want, backend[1], tol16=0.02)


@pytest.mark.parametrize("backend", [GPU16])
@pytest.mark.parametrize("name", ["all", "ragged"])
def test_kernel_for_any_width_in_16_bits(backend, name):
    sp, _ = ATTEND[name]
    for decode, seqs in ((False, [(90, 90), (120, 2)]), (True, [(33, 1), (150, 1)])):
        data, tables, rows = paged(sp, seqs, *backend, 16)
        got, want = run(sp, data, tables, rows, backend, 16, decode=decode, simple=True, sink=sinks(sp.heads))
        close(got, want, backend[1], tol16=0.02)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("win", [NO_WINDOW, 1, 64, 65, 150])
def test_one_key_among_hundreds(backend, decode, win):
    """A key that reaches the bound of the scores: far back, at page and tile borders, just inside and just outside the window."""
    sp = dataclasses.replace(spec(4, 2, 32, 48, win, cap=25.0), scale=0.3)
    for i in (511, 512, 700):
        for j in {0, 1, 63, 64, 255, 256, i - win, i - win + 1, i - 1, i} & set(range(i + 1)):
            data, tables, rows = paged(sp, [(i + 1, 1 if decode else 9)], *backend, 64, seed=i, noise=0.2)
            q, k, v = data[0]
            q[-1] = q[-1, :1]
            dirn = q[-1, 0, 0] / q[-1, 0, 0].norm()
            q[-1, :, 0] = (8.0 * dirn).to(torch.bfloat16).float()
            k[j, :, 0] = (60.0 * dirn).to(torch.bfloat16).float()
            v[j] = v[j] + 3.0
            got, want = run(sp, data, tables, rows, backend, 64, decode=decode, sink=sinks(4, 2.0))
            close(got[-1:], want[-1:], backend[1], tol16=0.02, tol32=1e-4)
            value = v[j].repeat_interleave(2, 0).double()
            assert (float((want[-1].view(4, 48) - value).abs().max()) < 0.05) == (i - j < win)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("decode", [False, True])
def test_sinks_far_above_and_far_below_the_scores(backend, decode):
    sp = spec(6, 2, 32, 32)
    data, tables, rows = paged(sp, [(90, 1 if decode else 90), (3, 1 if decode else 3)], *backend, 16)
    s = torch.tensor([-300.0, -20.0, 0.0, 4.0, 12.0, 300.0])
    got, want = run(sp, data, tables, rows, backend, 16, decode=decode, sink=s)
    assert bool((want.view(-1, 6, 32)[:, 5].abs() < 1e-9).all()) and bool(torch.isfinite(got).all())
    for h in range(6):     # every head on its own scale
        w = want.view(-1, 6, 32)[:, h]
        if float(w.abs().max()) > 1e-9:
            close(got.view(-1, 6, 32)[:, h], w, backend[1], tol16=0.02, tol32=5e-5)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("decode", [False, True])
def test_bounded_scores_over_their_whole_range(backend, decode):
    """Scores from far below minus the bound to far above it, and small ones; rising along the keys."""
    for cap, top in ((30.0, 90.0), (1.0, 0.01), (50.0, 24.0)):
        sp = dataclasses.replace(spec(2, 1, 16, 32, cap=cap), scale=1.0)
        data, tables, rows = paged(sp, [(300, 1 if decode else 300)], *backend, 64, noise=0.01)
        q, k, _ = data[0]
        q[..., 0] = 4.0
        k[..., 0] = torch.linspace(-top / 4, top / 4, 300).view(-1, 1, 1).to(torch.bfloat16).float()
        got, want = run(sp, data, tables, rows, backend, 64, decode=decode, sink=torch.tensor([0.5, 2.0]))
        close(got, want, backend[1], tol16=0.02, tol32=2e-4)


# -------------------------------------------------------------------------------------------------- routing
RULES = {"plain": (6, 2, 0, 0, 1, 1, 1.0, False), "identity": (7, 3, 2, 1, 3, 2, 2.5, True), "one-group": (12, 2, 4, 2, 4, 1, 0.7, True),
         "all-groups": (30, 8, 10, 0, 5, 5, 1.0, False), "many": (120, 4, 40, 3, 16, 3, 1.5, True), "only": (1, 1, 0, 1, 1, 1, 3.0, False),
         "mostly-identity": (2, 3, 6, 1, 2, 1, 1.0, True), "hundreds": (300, 6, 84, 0, 96, 5, 1.0, False)}


def routing_case(T, name, device, seed=7, skew=0.0):
    """(Scored, logits as a branch, plain logits [T, outputs (+ 1)], plain rule)"""
    E, top, identity, always, groups, keep, scale, gated = RULES[name]
    n = E + identity
    z = rand(T, n + gated, seed=seed, scale=1.5)
    z[:, :n] += skew * torch.arange(n)
    a = rand(T, n + gated, seed=seed + 1)
    correction = rand(n, seed=seed + 2, scale=0.1) - 0.2
    s = moe.Scored(correction.to(device), identity, groups, keep, scale, gated)
    return s, Branch(slabs=torch.stack([a, z - a]).to(device)), z, correction, {"top": top, "scale": scale, "groups": {"count": groups, "keep": keep}}


@pytest.mark.parametrize("backend", BACKENDS[:2])
@pytest.mark.parametrize("T", [1, 5, 128, 129, 300])
@pytest.mark.parametrize("name", list(RULES))
def test_scored_routing(backend, T, name):
    device, _ = backend
    E, top, identity, always, *_ = RULES[name]
    s, branch, z, correction, rule = routing_case(T, name, device)
    slots = torch.arange(T)
    if T > 2:
        slots[[0, T // 2]] = -1
    for f32 in ([False] if device == "cpu" else [False, True]):
        r = moe.route(branch, top, E, always, slots.to(device), f32=f32, scored=s)
        status(device)
        pos, weight, own = r.pos.cpu(), r.weight.cpu(), r.self_weight.cpu()
        owner = {}
        for e, first, count, _ in r.groups.cpu()[:int(r.n_groups[0])].tolist():
            assert 0 < count <= r.tile_rows
            owner |= {row: e for row in range(first, first + count)}
        used = pos[pos >= 0].tolist()
        assert sorted(used) == list(range(len(used))) == sorted(owner)
        for t in range(T):
            if slots[t] < 0:
                assert bool((pos[t] < 0).all()) and float(own[t]) == 0.0
                continue
            want = oracle.route(z[t, :E + identity].double(), correction.double(), rule)
            shared = float(torch.sigmoid(z[t, -1])) if s.always_gate else 1.0
            got = {owner[int(p)]: float(w) for p, w in zip(pos[t], weight[t]) if p >= 0}
            expected = {e: w for e, w in want if e < E} | {E + i: shared for i in range(always)}
            assert got.keys() == expected.keys() and all(abs(got[e] - expected[e]) < 2e-5 for e in expected), (t, got, expected)
            assert abs(float(own[t]) - sum(w for e, w in want if e >= E)) < 2e-5
            assert all(int(r.row_token[int(p)]) == t for p in pos[t] if p >= 0)


@pytest.mark.parametrize("backend", BACKENDS[:2])
def test_correction_and_groups_decide_and_do_not_weigh(backend):
    """A correction that turns the choice round; a group whose second best outscores every other group stays closed."""
    device, _ = backend
    z = torch.tensor([[3.0, 2.9, 0.0, 0.1, -1.0, 2.0]])
    for correction, groups, keep, want in (([0.0] * 6, 1, 1, (0, 1)), ([-1.0, 0, 0, 0, 0, 0], 1, 1, (1, 5)), ([0.0] * 6, 3, 1, (0, 1)),
                                           ([-1.0, -1.0, -0.9, -0.9, -2.0, -1.5], 3, 2, (0, 1)), ([-2.0, -2.0, -0.5, -0.6, -0.9, -0.4], 3, 1, (4, 5)),
                                           ([-2.0, -2.0, -0.5, -0.6, -0.9, -0.7], 3, 1, (2, 3))):
        s = moe.Scored(torch.tensor(correction).to(device), 0, groups, keep, 1.0)
        r = moe.route(Branch(slabs=z[None].to(device)), 2, 6, 0, torch.arange(1).to(device), scored=s)
        chosen = sorted(int(e) for e, *_ in r.groups.cpu()[:int(r.n_groups[0])])
        assert tuple(chosen) == want
        p = torch.softmax(z[0], 0)[list(want)]
        assert torch.allclose(r.weight.cpu().sort().values, (p / p.sum())[None].sort().values, atol=1e-6)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("T", [1, 17, 128, 300])
@pytest.mark.parametrize("name", ["identity", "one-group", "mostly-identity"])
def test_mixture_into_the_stream(backend, T, name):
    """Routed experts, the token's own row, a gated shared expert wider than the routed ones, then the norm around zero behind the
    sublayer and the one in front of the next."""
    device, dtype = backend
    E, top, identity, always, *_ = RULES[name]
    W, F, eps = 96, 48, 1e-4
    s, branch, z, correction, rule = routing_case(T, name, device, seed=31)
    x = rand(T, W, seed=3)
    gu, down = rand(E + always, 2 * F, W, seed=4, scale=W ** -0.5), rand(E + always, W, F, seed=5, scale=F ** -0.5)
    slots = torch.arange(T)
    r = moe.route(branch, top, E, always, slots.to(device), f32=dtype == torch.float32, scored=s)
    ff = moe.expert_ffn(x.to(device, dtype), r, gu.to(device, dtype), down.to(device, dtype))
    post, nxt = rand(W, seed=8, scale=0.3), rand(W, seed=9, scale=0.3)
    ff.post_norm = post.to(device, dtype)
    stream, n = x.clone().to(device), torch.empty((T, W), dtype=dtype, device=device)
    lat.stream_update(stream, W, eps, keep=True, a=ff, norm_weight=nxt.to(device, dtype), norm_out=n, norm_offset=1.0)
    status(device)
    want = x.double()
    for t in range(T):
        y = torch.zeros(W, dtype=torch.float64)
        shared = [(E + i, float(torch.sigmoid(z[t, -1].double())) if s.always_gate else 1.0) for i in range(always)]
        for e, weight in oracle.route(z[t, :E + identity].double(), correction.double(), rule):
            if e >= E:
                y += weight * x[t].double()
            else:
                shared.append((e, weight))
        for e, weight in shared:
            h = gu[e].double() @ x[t].double()
            y += weight * (down[e].double() @ (oracle.silu(h[:F]) * h[F:]))
        want[t] += oracle.norm_around_zero(y, post.double(), eps)
    close(stream, want, dtype, tol16=0.015)
    close(n, oracle.norm_around_zero(want, nxt.double(), eps), dtype, tol16=0.02)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("width,T", [(64, 3), (1200, 300), (4112, 4)])
def test_own_row_and_scaled_embedding(backend, width, T):
    """The stream's own row in a branch, for one and for several column groups per thread; a scaled embedding lookup."""
    device, dtype = backend
    x0, slabs, post = rand(T, width, seed=1), rand(2, T, width, seed=2), rand(width, seed=3, scale=0.3)
    own = rand(T, seed=4).abs()
    x = x0.clone().to(device)
    lat.stream_update(x, width, 2e-3, keep=True, norm_offset=1.0,
                      a=Branch(slabs=slabs.to(device), post_norm=post.to(device, dtype), self_weight=own.to(device)))
    want = x0.double() + oracle.norm_around_zero(slabs.double().sum(0) + own.double()[:, None] * x0.double(), post.double(), 2e-3)
    close(x, want, torch.float32, tol32=3e-6)
    table, ids = rand(11, width, seed=5), torch.arange(T) % 11
    raw = torch.empty((T, width), dtype=dtype, device=device)
    lat.stream_update(x, width, 1e-5, keep=False, ids=ids.to(device), table=table.to(device, dtype), embed_mult=2.7, raw_out=raw)
    close(x, table[ids].double() * 2.7, torch.float32, tol32=1e-6)
    close(raw, table[ids].double() * 2.7, dtype)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("T", [3, 140, 600])
@pytest.mark.parametrize("M,K", [(272, 96), (1024, 64), (97, 80)])
def test_scaled_and_decay_sections_in_32_bit(backend, T, M, K):
    """Sections of a stacked projection with fp32 output: a scale (logits), and decays; few tokens, and enough for the persistent form."""
    device, dtype = backend
    x, w, bias = rand(T, K, seed=1), rand(M, K, seed=2, scale=K ** -0.5), rand(M, seed=3)
    y = x.double() @ w.double().T
    args = x.to(device, dtype), w.to(device, dtype)
    got = lat.linear_sections(*args, lat.Sections([(M, 2.5, None)]), out_f32=True)
    close(got, y * 2.5, dtype, tol16=1e-5)
    first = M // 2 // 16 * 16
    got = lat.linear_sections(*args, lat.Sections([(first, 1.0, "decay"), (M - first, -0.5, None)]), bias=bias.to(device, dtype), out_f32=True)
    close(got[:, :first], torch.exp(-torch.exp(y[:, :first] + bias[:first].double())), dtype, tol16=1e-5)
    close(got[:, first:], -0.5 * y[:, first:] + bias[first:].double(), dtype, tol16=1e-5)
