"""Mixture of experts and the norm behind a sublayer, each against the plain float64 statement.  CPU statements, and the
kernels on a B200."""

import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import dolidra_oracle as oracle  # noqa: E402
from op_helpers import BACKENDS, close, rand  # noqa: E402

from prism_infer_b200 import ops  # noqa: E402
from prism_infer_b200.ops import latent as lat  # noqa: E402
from prism_infer_b200.ops import moe  # noqa: E402
from prism_infer_b200.ops.latent import Branch  # noqa: E402


def logits_of(T, E, seed, device):
    z = rand(T, E, seed=seed, scale=2.0)
    a = rand(T, E, seed=seed + 1)
    return z, Branch(slabs=torch.stack([a, z - a]).to(device))


def check_routing(r, z, top, always, live):
    """Weights and experts of every token, and the table of tiles: together they name every pair once."""
    T, E = z.shape
    pos, weight, groups = r.pos.cpu(), r.weight.cpu(), r.groups.cpu()[:int(r.n_groups[0])].tolist()
    assert not bool((pos[~live] >= 0).any())
    used = pos[live].reshape(-1)
    assert sorted(used.tolist()) == list(range(len(used)))
    expert_of = {}
    for e, first, count, _ in groups:
        assert 0 < count <= r.tile_rows
        for row in range(first, first + count):
            assert row not in expert_of
            expert_of[row] = e
    assert sorted(expert_of) == sorted(used.tolist())
    chosen = oracle.route(z.double(), torch.eye(E, dtype=torch.float64), top)
    for t in range(T):
        if not live[t]:
            continue
        got = {expert_of[int(p)]: float(w) for p, w in zip(pos[t], weight[t])}
        want = dict(chosen[t]) | {E + s: 1.0 for s in range(always)}
        assert got.keys() == want.keys()
        assert all(abs(got[e] - want[e]) < 1e-5 for e in want)
        assert all(int(r.row_token[int(p)]) == t for p in pos[t])


@pytest.mark.parametrize("backend", BACKENDS[:2])
@pytest.mark.parametrize("T", [1, 5, 64, 128, 129, 300])
@pytest.mark.parametrize("E,top,always", [(6, 2, 1), (1, 1, 0), (40, 8, 2), (7, 7, 0), (130, 3, 1)])
def test_routing(backend, T, E, top, always):
    device, _ = backend
    z, b = logits_of(T, E, 7, device)
    slots = torch.arange(T)
    if T > 2:
        slots[[0, T // 2]] = -1
    for f32 in ([False] if device == "cpu" else [False, True]):
        r = moe.route(b, top, E, always, slots.to(device), f32=f32)
        check_routing(r, z, top, always, slots >= 0)


@pytest.mark.parametrize("backend", BACKENDS[:2])
def test_equal_logits_go_to_the_lowest_experts(backend):
    device, _ = backend
    z = torch.zeros(3, 50)
    z[1, 40:] = 1.0
    r = moe.route(Branch(slabs=z[None].to(device)), 3, 50, 0, torch.arange(3).to(device))
    groups = r.groups.cpu()[:int(r.n_groups[0])].tolist()
    assert [(e, n) for e, _, n, _ in groups] == [(0, 2), (1, 2), (2, 2), (40, 1), (41, 1), (42, 1)]


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("T", [1, 3, 17, 40, 128, 130, 700])
@pytest.mark.parametrize("E,top,always,W,F,skew", [(6, 2, 1, 96, 48, False), (1, 1, 0, 64, 16, False), (40, 4, 2, 112, 208, False),
                                                   (9, 3, 0, 320, 144, True)])
def test_expert_feed_forwards(backend, T, E, top, always, W, F, skew):
    """Routed and always-on experts through the grouped projections and the weighted sum in the residual stream; skew: every
    token picks the same experts."""
    device, dtype = backend
    z, b = logits_of(T, E, 11, device)
    if skew:
        z = z[:1].expand(T, E).contiguous()
        b = Branch(slabs=z[None].to(device))
    x = rand(T, W, seed=3)
    gu, down = rand(E + always, 2 * F, W, seed=4, scale=W ** -0.5), rand(E + always, W, F, seed=5, scale=F ** -0.5)
    slots = torch.arange(T)
    if T > 2:
        slots[1] = -1
    r = moe.route(b, top, E, always, slots.to(device), f32=dtype == torch.float32)
    got = moe.expert_ffn(x.to(device, dtype), r, gu.to(device, dtype), down.to(device, dtype))
    want = torch.zeros(T, W, dtype=torch.float64)
    chosen = oracle.route(z.double(), torch.eye(E, dtype=torch.float64), top)
    for t in range(T):
        if slots[t] >= 0:
            for e, weight in chosen[t] + [(E + s, 1.0) for s in range(always)]:
                h = x[t].double() @ gu[e].double().T
                want[t] += weight * ((oracle.silu(h[:F]) * h[F:]) @ down[e].double().T)
    stream = torch.zeros((T, W), device=device)
    lat.stream_update(stream, W, 1e-5, keep=False, a=got, raw_out=torch.empty((T, W), dtype=dtype, device=device))
    close(stream, want, dtype, tol16=0.015)
    assert T <= 2 or bool((stream[1] == 0).all())
    if device != "cpu":
        from prism_infer_b200.ops import native

        native.check_status()


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("act", ["silu", "gelu_tanh"])
@pytest.mark.parametrize("T", [1, 20, 100, 200, 600])
def test_gated_unit(backend, act, T):
    device, dtype = backend
    K, F = 136, 208
    x, w = rand(T, K, seed=1), rand(2 * F, K, seed=2, scale=2 * K ** -0.5)
    h = x.double() @ w.double().T
    fn = oracle.silu if act == "silu" else oracle.gelu_tanh
    close(ops.gate_up_glu(x.to(device, dtype), w.to(device, dtype), act), fn(h[:, :F]) * h[:, F:], dtype)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("width,padded", [(64, 64), (75, 80), (1200, 1200), (4100, 4112)])
@pytest.mark.parametrize("pairs", [False, True])
def test_norm_behind_a_sublayer(backend, width, padded, pairs):
    """The branch over its own root mean square times a weight, added to the stream, and the weighted norm that follows; the
    branch as slabs or as the weighted sum of pair rows (one of them absent)."""
    device, dtype = backend
    T, K, eps = 4, 3, 2e-3

    def wide(t):
        return torch.nn.functional.pad(t, (0, padded - width))

    x0, post, w = wide(rand(T, width, seed=1)), wide(rand(width, seed=2)), wide(rand(width, seed=3))
    slabs = wide(rand(2, T * K if pairs else T, width, seed=4))
    pos = torch.tensor([[3, 0, 11], [1, 2, -1], [7, 8, 4], [5, 6, 10]], dtype=torch.int32)
    weight = rand(T, K, seed=5).abs()
    y = slabs.double().sum(0)
    if pairs:
        y = torch.stack([sum(float(weight[t, k]) * y[int(pos[t, k])] for k in range(K) if pos[t, k] >= 0) for t in range(T)])
    want = x0.double()
    want[:, :width] += oracle.norm(y[:, :width], post[:width].double(), eps)
    x, n = x0.to(device), torch.full((T, padded), 9.0, dtype=dtype, device=device)
    branch = Branch(slabs=slabs.to(device), post_norm=post.to(device, dtype), pos=pos.to(device) if pairs else None,
                    weight=weight.to(device) if pairs else None)
    lat.stream_update(x, width, eps, keep=True, a=branch, norm_weight=w.to(device, dtype), norm_out=n)
    close(x, want, torch.float32, tol32=3e-6)
    close(n, wide(oracle.norm(want[:, :width], w[:width].double(), eps)), dtype)
    rows = rand(T, padded, seed=8).to(dtype)  # rows of the compute type, without a weight on the norm that follows
    rows[:, width:] = 0
    x, want = x0.to(device), x0.double()
    want[:, :width] += oracle.norm(rows.double()[:, :width], post[:width].double(), eps)
    lat.stream_update(x, width, eps, keep=True, a=Branch(rows=rows.to(device), post_norm=post.to(device, dtype)), norm_out=n)
    close(x, want, torch.float32, tol32=3e-6)
    close(n, wide(oracle.rms(want[:, :width], eps)), dtype)
