"""Time mixing with a matrix state per head: blends with the previous token, decays, the recurrence in prompts, portions and
steps, the slots and versions of the state; against the plain float64 statement.  CPU statements, and the kernels on a B200."""

import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import bokorax_oracle as oracle  # noqa: E402
from op_helpers import BACKENDS, GPU16, GPU32, close, rand  # noqa: E402

from prism_infer_b200.ops import recurrent as rec  # noqa: E402

# heads, channels, rank of the decay, width of the rows
SIZES = {"small": (3, 24, 12, 96), "ragged": (5, 13, 5, 75), "tile": (2, 64, 64, 128), "two-tiles": (3, 72, 33, 160), "wide": (2, 128, 40, 144),
         "widest": (1, 256, 24, 96), "odd": (2, 200, 3, 64), "many": (9, 16, 7, 64)}
EPS = 2e-4


def up(n):
    return -(-n // 16) * 16


class Mixer:
    """Weights of one mixer, plain (for the oracle, with an identity as output projection) and packed."""

    def __init__(self, name, backend, slots=5, slow=False):
        H, d, R, W = SIZES[name]
        self.H, self.d, self.W, self.backend = H, d, W, backend
        device, dtype = backend
        C = H * d
        p = {"mu." + s: rand(W, seed=i).abs().clamp_max(1.0) for i, s in enumerate("rkvgw")}
        p |= {s: rand(C, W, seed=10 + i, scale=1.2 * W ** -0.5) for i, s in enumerate("rkvg")}
        p |= {"w1": rand(R, W, seed=20, scale=2 * W ** -0.5), "w2": rand(C, R, seed=21, scale=(0.1 if slow else 1.0) * R ** -0.5),
              "w0": torch.full((C,), -7.0) if slow else rand(C, seed=22) - 1.5, "u": rand(H, d, seed=23), "norm": 1.0 + 0.2 * rand(C, seed=24)}
        p["norm"] = p["norm"].to(torch.bfloat16).float()
        self.w = {k: v.double() for k, v in p.items()} | {"o": torch.eye(C, dtype=torch.float64)}
        self.spec = s = rec.TimeMixSpec(H, d, up(R), up(W), EPS)

        def z(*shape):
            return torch.zeros(shape, dtype=dtype, device=device)

        m = rec.TimeMixWeights(z(5, s.width), z(4, s.cols, s.width), z(s.rank, s.width), z(s.cols, s.rank), z(s.cols), z(s.cols), z(s.cols))
        for i, n in enumerate("rkvgw"):
            m.mu[i, :W] = p["mu." + n].to(device, dtype)
        for i, n in enumerate("rkvg"):
            m.rkvg[i].view(H, s.n, s.width)[:, :d, :W] = p[n].view(H, d, W).to(device, dtype)
        m.w1[:R, :W] = p["w1"].to(device, dtype)
        m.w2.view(H, s.n, -1)[:, :d, :R] = p["w2"].view(H, d, R).to(device, dtype)
        for n in ("w0", "u", "norm"):
            getattr(m, n).view(H, s.n)[:, :d] = p[n].reshape(H, d).to(device, dtype)
        self.packed = m
        self.cache = rec.StateCache([8, s.carry + s.width], slots, device)
        for i in range(2):
            self.cache.layer(i).fill_(1e4)     # what an earlier owner left behind

    def rows(self, T, seed):
        return rand(T, self.W, seed=seed)

    def want(self, x):
        return oracle.time_mix(x.double(), self.w, "", {"heads": self.H, "dim": self.d}, EPS, None)[0]

    def step(self, parts, *, decode=False):
        """parts: (rows, slot, tokens before); -> outputs [tokens, H * d] without padding."""
        device, _ = self.backend
        x = torch.nn.functional.pad(torch.cat([p[0] for p in parts]), (0, self.spec.width - self.W)).to(device)
        lens = [p[0].shape[0] for p in parts]
        cu = None if decode else torch.tensor([0] + lens).cumsum(0).to(torch.int32).to(device)
        view = rec.StateView(self.cache, 1, torch.tensor([p[1] for p in parts], dtype=torch.int32).to(device),
                             torch.tensor([n + p[2] for n, p in zip(lens, parts)], dtype=torch.int32).to(device), cu)
        y = rec.time_mix(x, self.spec, self.packed, view)
        if device != "cpu":
            from prism_infer_b200.ops import native

            native.check_status()
        y = y.float().cpu().view(-1, self.H, self.spec.n)
        assert bool((y[:, :, self.d:] == 0).all())
        return y[:, :, :self.d].flatten(1)

    def near(self, got, want, tol16=0.03):
        close(got, want, self.backend[1], tol16=tol16, tol32=1e-4)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", list(SIZES))
def test_whole_sequence(backend, name):
    m = Mixer(name, backend)
    for T in (1, 2, 15, 16, 17, 90):
        x = m.rows(T, 100 + T)
        m.near(m.step([(x, 3, 0)]), m.want(x))


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", list(SIZES))
def test_token_by_token_equals_the_sequence(backend, name):
    m = Mixer(name, backend)
    x = m.rows(40, 3)
    got = torch.cat([m.step([(x[i:i + 1], 1, i)], decode=True) for i in range(40)])
    m.near(got, m.want(x))


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("sizes", [[2], [3], [1, 2], [16, 4], [17, 15], [33, 1, 1], [5, 40]])
def test_portions(backend, sizes):
    """Cut anywhere; portions of odd and even length, so that a version is read and written by the same step."""
    m = Mixer("ragged", backend)
    x = m.rows(75, 4)
    at, i, got = 0, 0, []
    while at < 75:
        n = min(sizes[i % len(sizes)], 75 - at)
        got.append(m.step([(x[at:at + n], 2, at)], decode=n == 1 and i % 2 == 1 and at > 0))
        at, i = at + n, i + 1
    m.near(torch.cat(got), m.want(x))


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", ["small", "two-tiles"])
def test_batches_and_reused_slots(backend, name):
    """Portions of some sequences beside single tokens of others, each as if alone; slots handed on to new sequences."""
    m = Mixer(name, backend)
    xs = [m.rows(n, 50 + n) for n in (61, 30, 45, 20)]
    out = [[] for _ in xs]
    at = [0] * 4
    for step in ([(0, 30), (1, 2)], [(0, 1), (1, 15), (2, 40)], [(2, 2), (0, 1)], [(1, 13), (0, 29), (2, 3)]):
        parts = [(xs[r][at[r]:at[r] + n], r, at[r]) for r, n in step]
        y, base = m.step(parts), 0
        for r, n in step:
            out[r].append(y[base:base + n])
            base, at[r] = base + n, at[r] + n
    assert at[:3] == [61, 30, 45]
    for r in range(3):
        m.near(torch.cat(out[r]), m.want(xs[r]))
    m.near(m.step([(xs[3], 1, 0)]), m.want(xs[3]))      # slot 1 once more
    one = m.rows(1, 9)
    m.near(m.step([(one, 0, 0)], decode=True), m.want(one))


@pytest.mark.parametrize("backend", BACKENDS)
def test_a_repeated_step_reads_what_it_read_before(backend):
    """A step one token ahead leaves the state it started from alone, for single tokens and for portions of odd length."""
    m = Mixer("tile", backend)
    x = m.rows(30, 6)
    got = [m.step([(x[:9], 4, 0)])]
    other = m.rows(7, 7)
    for i in range(9, 14):
        m.step([(other[:1], 4, i)], decode=True)         # ran ahead with another token, discarded
        got.append(m.step([(x[i:i + 1], 4, i)], decode=True))
    m.step([(other, 4, 14)])
    got.append(m.step([(x[14:21], 4, 14)]))
    got.append(m.step([(x[21:], 4, 21)]))
    m.near(torch.cat(got), m.want(x))


@pytest.mark.parametrize("backend", BACKENDS)
def test_rows_without_a_slot(backend):
    """Padding rows give zeros and touch no state."""
    m = Mixer("small", backend)
    x = m.rows(3, 8)
    before = m.cache.layer(1).clone()
    y = m.step([(x[:1], 2, 0), (x[1:2], -1, 0), (x[2:], 0, 0)], decode=True)
    m.near(y[[0, 2]], torch.cat([m.want(x[:1]), m.want(x[2:])]))
    assert bool((y[1] == 0).all())
    y = m.step([(x, -1, 4), (x, 3, 0)])
    assert bool((y[:3] == 0).all())
    m.near(y[3:], m.want(x))
    after = m.cache.layer(1)
    for slot in (1, 4):
        assert torch.equal(after[slot], before[slot])
    assert torch.equal(after[2, 0], before[2, 0]) and not torch.equal(after[2, 1], before[2, 1])
    assert bool((m.cache.layer(0) == 1e4).all())


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("decode", [False, True])
def test_a_far_token_is_remembered(backend, decode):
    """Slow decay and one key that stands out: its value dominates hundreds of tokens later, and not before."""
    m = Mixer("tile", backend, slow=True)
    H, d = m.H, m.d
    x = 0.2 * m.rows(401, 12)
    k_dir = torch.linalg.lstsq(torch.cat([m.w["k"], m.w["r"]]), torch.cat([torch.ones(H * d), 0.0 * torch.ones(H * d)]).double()[:, None]).solution[:, 0]
    x[20] = (30.0 * k_dir / k_dir.norm()).float().to(torch.bfloat16).float()
    want = m.want(x)
    if decode:
        got = torch.cat([m.step([(x[:300], 0, 0)])] + [m.step([(x[i:i + 1], 0, i)], decode=True) for i in range(300, 401)])
    else:
        got = torch.cat([m.step([(x[:200], 0, 0)]), m.step([(x[200:], 0, 200)])])
    m.near(got, want, tol16=0.06)
    y = x.clone()
    y[20] = x[21]
    assert float((m.want(y)[400] - want[400]).abs().max()) > 0.2 * float(want[400].abs().max())


@pytest.mark.parametrize("backend", [GPU32, GPU16])
@pytest.mark.parametrize("T,C,R,S", [(1, 16, 16, 1), (70, 144, 48, 3), (129, 256, 64, 2), (64, 128, 128, 1), (600, 400, 208, 2)])
def test_decays(backend, T, C, R, S):
    """From rates that forget at once to rates that forget nothing in thousands of tokens; close to 32-bit in both types."""
    device, dtype = backend
    z, w2, w0 = rand(S, T, R, seed=1, scale=1.0), rand(C, R, seed=2, scale=2 * R ** -0.5), torch.linspace(-9.0, 3.0, C).to(torch.bfloat16).float()
    w = rec.TimeMixWeights(*(torch.zeros(1),) * 3, w2.to(device, dtype), w0.to(device, dtype), *(torch.zeros(1),) * 2)
    got = rec.decays(z.to(device), w).double().cpu()
    rate = torch.exp(torch.tanh(z.double().sum(0)) @ w2.double().T + w0.double())
    assert float((got - torch.exp(-rate)).abs().max()) < (2e-6 if dtype == torch.float32 else 1e-4)
    slow = rate < 0.1
    assert float(((-torch.log(got) - rate).abs() / rate)[slow & (rate > 1e-2)].max()) < (1e-4 if dtype == torch.float32 else 1e-3)
    from prism_infer_b200.ops import native

    native.check_status()


@pytest.mark.parametrize("backend", [GPU32, GPU16])
def test_long_prompts(backend):
    """More tokens than the small-step projections take, several sequences, ragged token blocks."""
    m = Mixer("two-tiles", backend)
    xs = [m.rows(n, 70 + n) for n in (333, 1, 130, 16)]
    y = m.step([(x, s, 0) for s, x in enumerate(xs)])
    m.near(y, torch.cat([m.want(x) for x in xs]))


def test_slots_move_between_caches():
    a, b = rec.StateCache([6, 9], 3, "cpu"), rec.StateCache([6, 9], 2, "cpu")
    for i in range(2):
        a.layer(i).copy_(torch.arange(a.layer(i).numel()).view(a.layer(i).shape))
    b.copy_slot(a, 2, 1)
    assert torch.equal(b.layer(0)[1], a.layer(0)[2]) and torch.equal(b.layer(1)[1], a.layer(1)[2]) and bool((b.layer(1)[0] == 0).all())
    assert a.bytes() == 3 * 2 * 15 * 4
