"""Ops of the Fosulix family, each against the plain float64 statement: rotary frequencies by turns, latent rows with a rotated key
part, windowed latent attention in both forms, the short convolution and the forget rule with their state slots, the depth average,
routing by sigmoid scores and bounded experts.  CPU statements, and the kernels on a B200."""

import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import fosulix_oracle as oracle  # noqa: E402
from op_helpers import BACKENDS, GPU16, close, rand  # noqa: E402

from prism_infer_b200 import ops  # noqa: E402
from prism_infer_b200.models.architecture import LatentAttentionArch, RotaryArch  # noqa: E402
from prism_infer_b200.ops import latent as lat  # noqa: E402
from prism_infer_b200.ops import moe  # noqa: E402
from prism_infer_b200.ops import recurrent as rec  # noqa: E402
from prism_infer_b200.ops.latent import Branch  # noqa: E402

EPS = 2e-4
NO_WINDOW = lat.NO_WINDOW


def up(n, to=16):
    return -(-n // to) * to


def status(device):
    if device != "cpu":
        from prism_infer_b200.ops import native

        native.check_status()


# ------------------------------------------------------------------------------------------------ rotation
@pytest.mark.parametrize("dims,base,factor,original,fast,slow", [(16, 9000.0, 4.0, 64, 8.0, 1.0), (64, 1e6, 32.0, 4096, 32.0, 1.0), (2, 500.0, 2.0, 30, 1.0, 0.5),
                                                                 (24, 300.0, 8.0, 128, 900.0, 0.001), (12, 7000.0, 3.0, 96, 2.0, 2.0)])
def test_frequencies_by_turns(dims, base, factor, original, fast, slow):
    """Ramps of several lengths, also none, and ends past the first and the last pair."""
    rot = {"base": base, "dims": dims, "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}}
    f, size = oracle.frequencies(rot)
    arch = RotaryArch(base, dims, factor=factor, original=original, fast=fast, slow=slow)
    assert torch.allclose(torch.tensor(arch.inv_freq(), dtype=torch.float64), f, rtol=1e-12) and abs(arch.amplitude - size) < 1e-12
    plain = RotaryArch(base, dims)
    assert plain.amplitude == 1.0 and torch.allclose(torch.tensor(plain.inv_freq(), dtype=torch.float64), oracle.frequencies({"base": base, "dims": dims})[0])


ROT = {"base": 400.0, "scaling": {"factor": 3.0, "original": 80, "fast": 5.0, "slow": 1.0}}


def arch_of(heads, dim, vdim, rank, q_rank, rot, window=NO_WINDOW):
    s = ROT["scaling"]
    return LatentAttentionArch(heads, dim, vdim, rank, 1.3 * (dim + rot) ** -0.5, q_rank=q_rank, rot_dim=rot, window=window,
                               rot=RotaryArch(ROT["base"], rot, factor=s["factor"], original=s["original"], fast=s["fast"], slow=s["slow"]))


def weights_of(m, backend, seed=0, own=True):
    """Plain weights, and packed ones."""
    device, dtype = backend
    w = {"dq.norm": 1 + 0.3 * rand(m.q_rank, seed=seed + 1), "dkv.norm": 1 + 0.3 * rand(m.kv_rank, seed=seed + 2),
         "uk": rand(m.heads * m.dim, m.kv_rank, seed=seed + 3, scale=m.kv_rank ** -0.5), "uv": rand(m.heads * m.vdim, m.kv_rank, seed=seed + 4, scale=m.kv_rank ** -0.5)}
    w = {k: v.to(torch.bfloat16).float() for k, v in w.items()}
    z = lambda *s: torch.zeros(s, dtype=dtype, device=device)  # noqa: E731
    rot = lat.Rotary(torch.tensor(m.rot.inv_freq(), dtype=torch.float64).float().to(device), m.rot_dim, m.rot_start, m.row_rot_start, m.rot.amplitude)
    lw = lat.LatentWeights(m.heads, m.dq, m.dv, m.kv_rank, m.scale, z(m.row_rot_start) if own else None, z(m.heads * (m.dq + m.dv), m.cache_row), rot,
                           m.window, m.q_rank, z(up(m.q_rank)))
    lw.connect_rotary()
    lw.q_norm[:m.q_rank] = w["dq.norm"].to(device, dtype)
    if own:
        lw.norm[:m.kv_rank] = w["dkv.norm"].to(device, dtype)
    lw.uk.view(m.heads, m.dq, -1)[:, :m.dim, :m.kv_rank] = w["uk"].view(m.heads, m.dim, -1).to(device, dtype)
    lw.uv.view(m.heads, m.dv, -1)[:, :m.vdim, :m.kv_rank] = w["uv"].view(m.heads, m.vdim, -1).to(device, dtype)
    return {k: v.double() for k, v in w.items()}, lw


def as_branch(x, source, backend, splits=3):
    """fp32 ``x`` as slabs whose sum it is, or as rows of the compute type."""
    device, dtype = backend
    if source == "rows":
        return Branch(rows=x.to(device, dtype))
    parts = [rand(*x.shape, seed=91 + i) for i in range(splits - 1)]
    return Branch(slabs=torch.stack(parts + [x - sum(parts)]).to(device))


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("source", ["slabs", "rows"])
@pytest.mark.parametrize("T,rank,q_rank,rot", [(1, 56, 72, 12), (7, 21, 19, 6), (3, 64, 48, 2), (300, 512, 1536, 64), (5, 700, 33, 60)])
def test_latent_rows(backend, source, T, rank, q_rank, rot):
    """Both norms, the rotated key part, padding, slots that are skipped; a layer that reads another's rows has only queries."""
    if source == "slabs" and backend[0] != "cpu" and T > 256:
        T = 200
    device, dtype = backend
    m = arch_of(2, 8, 8, rank, q_rank, rot)
    w, lw = weights_of(m, backend)
    Q, C = up(q_rank), m.row_rot_start
    y = torch.zeros(T, Q + C + up(rot))
    q, c, k = rand(T, q_rank, seed=5), rand(T, rank, seed=6), rand(T, rot, seed=7)
    y[:, :q_rank], y[:, Q:Q + rank], y[:, Q + C:Q + C + rot] = q, c, k
    cache = ops.KVCache(2, 40, 1, 16, m.cache_row, ops.KV_BF16, device, dtype=dtype, planes=1, rows=(64, m.cache_row))
    cache.token_rows(1).fill_(5.0)
    slots = torch.randperm(40 * 16, generator=torch.Generator().manual_seed(1))[:T]
    slots[T // 2] = -1
    pos = torch.arange(T) * 3 + 11
    got = lat.latent_prepare(as_branch(y, source, backend), lw, EPS, pos.to(torch.int32).to(device), slots.to(device), cache, 1)
    close(got[:, :q_rank], oracle.rms(q.double(), EPS) * w["dq.norm"], dtype)
    assert bool((got[:, q_rank:] == 0).all())
    turned = torch.cat([oracle.rotate(k[t:t + 1, None].double(), {**ROT, "dims": rot}, int(pos[t]))[:, 0] for t in range(T)])
    rows = cache.token_rows(1).reshape(-1, m.cache_row).float().cpu()
    live = slots >= 0
    close(rows[slots[live]][:, :rank], (oracle.rms(c.double(), EPS) * w["dkv.norm"])[live], dtype) if live.any() else None
    if live.any():
        close(rows[slots[live]][:, C:C + rot], turned[live], dtype, tol32=4e-5)
        assert bool((rows[slots[live]][:, rank:C] == 0).all()) and bool((rows[slots[live]][:, C + rot:] == 0).all())
    untouched = torch.ones(40 * 16, dtype=torch.bool)
    untouched[slots[live]] = False
    assert bool((rows[untouched] == 5.0).all())
    _, alone = weights_of(m, backend, own=False)
    again = lat.latent_prepare(as_branch(y[:, :Q].contiguous(), source, backend), alone, EPS, pos.to(torch.int32).to(device), slots.to(device), cache, 1)
    close(again, got.cpu(), dtype)
    assert torch.equal(cache.token_rows(1).reshape(-1, m.cache_row).float().cpu(), rows)
    status(device)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("source", ["slabs", "rows"])
def test_queries_are_turned(backend, source):
    device, dtype = backend
    m = arch_of(3, 13, 8, 32, 16, 6)
    _, lw = weights_of(m, backend)
    x, pos = torch.zeros(9, 3, m.dq), torch.tensor([0, 1, 2, 77, 300, 5, 5, 1000, 64])
    x[..., :13], x[..., m.rot_start:m.rot_start + 6] = rand(9, 3, 13, seed=1), rand(9, 3, 6, seed=2)
    got = lat.rotate_queries(as_branch(x.view(9, -1), source, backend), lw, pos.to(torch.int32).to(device)).view(9, 3, m.dq)
    want = x.double()
    for t in range(9):
        want[t, :, m.rot_start:m.rot_start + 6] = oracle.rotate(x[t:t + 1, :, m.rot_start:m.rot_start + 6].double(), {**ROT, "dims": 6}, int(pos[t]))[0]
    close(got, want, dtype, tol32=5e-5)
    status(device)


# --------------------------------------------------------------------------------------- windowed attention
class Scene:
    """Sequences whose rows are in a paged cache (their last ``new`` tokens included) and the new tokens' queries in hand.

    ``lookups``: sequence -> position of the key that its last query is made to look at: the query is that key, scaled, so that its
    score stands out among all others."""

    def __init__(self, backend, m, page, lens, new, lookups=None, seed=0):
        device, dtype = backend
        self.m, self.backend, self.lens, self.new, self.page = m, backend, lens, new, page
        w, self.lw = weights_of(m, backend, seed)
        S, R, r, H, d = len(lens), m.kv_rank, m.rot_dim, m.heads, m.dim
        per = [-(-n // page) + 1 for n in lens]
        order = torch.randperm(sum(per) + 2, generator=torch.Generator().manual_seed(seed + 9)).to(torch.int32)
        table = torch.full((S, max(per)), -1, dtype=torch.int32)
        self.cache = ops.KVCache(2, sum(per) + 2, 1, page, m.cache_row, ops.KV_BF16, device, dtype=dtype, planes=1, rows=(64, m.cache_row))
        pages = self.cache.token_rows(1)
        pages.normal_()                                    # what earlier owners left behind
        self.positions, self.q, want = [], [], []
        at = 0
        for s, (n, k) in enumerate(zip(lens, new)):
            table[s, :per[s]] = order[at:at + per[s]]
            at += per[s]
            c, kr = rand(n, R, seed=seed + 20 + s).to(torch.bfloat16).float(), rand(n, r, seed=seed + 40 + s)
            row = torch.zeros(n, m.cache_row)
            row[:, :R], row[:, m.row_rot_start:m.row_rot_start + r] = c, kr
            for p in range(n):
                pages[int(table[s, p // page]), p % page] = row[p].to(device, dtype)
            keys = torch.cat([(c.double() @ w["uk"].T).view(n, H, d), kr.double()[:, None].expand(n, H, r)], -1)
            q = rand(k, H, d + r, seed=seed + 60 + s)
            if lookups and s in lookups:
                aim = keys[lookups[s]] / keys[lookups[s]].pow(2).sum(-1, keepdim=True) * 25.0 / m.scale
                q[-1] = aim.float().to(torch.bfloat16).float()
            # what the kernels rotate themselves is stored turned back
            first, turned = n - k, q.double()
            raw = q.clone()
            f, size = oracle.frequencies({**ROT, "dims": r})
            for t in range(k):
                for i in range(r // 2):
                    a = -float((first + t) * f[i])
                    cs, sn = torch.cos(torch.tensor(a)).item() / size, torch.sin(torch.tensor(a)).item() / size
                    u, v = q[t, :, d + 2 * i].clone(), q[t, :, d + 2 * i + 1].clone()
                    raw[t, :, d + 2 * i], raw[t, :, d + 2 * i + 1] = u * cs - v * sn, v * cs + u * sn
            if dtype == torch.bfloat16:                    # in 16 bits the stored query is what counts
                raw = raw.to(torch.bfloat16).float()
                turned = torch.cat([raw[..., :d].double(), oracle.rotate(raw[..., d:].double(), {**ROT, "dims": r}, first)], -1)
            padded = torch.zeros(k, H, m.dq)
            padded[..., :d], padded[..., m.rot_start:m.rot_start + r] = raw[..., :d], raw[..., d:]
            self.q.append(padded.view(k, -1))
            self.positions += list(range(first, n))
            v = (c.double() @ w["uv"].T).view(n, H, m.vdim)
            want.append(oracle.attend(turned, keys, v, m.scale, window=m.window, first=first))
        self.want, self.table = torch.cat(want), table.to(device)
        self.kv_lens = torch.tensor(lens, dtype=torch.int32).to(device)

    def run(self, form, nsplit=0):
        device, dtype = self.backend
        m, q = self.m, Branch(rows=torch.cat(self.q).to(device, dtype))
        if form == "slabs":
            q = as_branch(torch.cat(self.q), "slabs", self.backend)
        pos = torch.tensor(self.positions, dtype=torch.int32).to(device)
        T = len(self.positions)
        if all(k == 1 for k in self.new) and form != "expanded":
            got = lat.latent_attention_absorbed(q, None, None, self.lw, EPS, torch.zeros(T, dtype=torch.int64).to(device), self.cache, 1, self.table,
                                                self.kv_lens, positions=pos, nsplit=nsplit)
        else:
            cu = torch.tensor([0] + self.new).cumsum(0).to(torch.int32).to(device)
            if form == "expanded":
                plan = lat.ExpandPlan.make(list(zip(self.new, self.lens)), m.window, self.page, self.table.shape[1], device)
                got = lat.latent_attention_windowed(lat.rotate_queries(q, self.lw, pos), self.lw, self.cache, 1, self.table, self.kv_lens, cu, max(self.new), plan)
            else:
                got = lat.latent_attention_absorbed(q, None, None, self.lw, EPS, torch.zeros(T, dtype=torch.int64).to(device), self.cache, 1, self.table,
                                                    self.kv_lens, cu_seqlens_q=cu, max_q_len=max(self.new), positions=pos, nsplit=nsplit)
        status(device)
        got = got.view(T, m.heads, m.dv)
        assert bool((got[..., m.vdim:] == 0).all())
        return got[..., :m.vdim]

    def check(self, form, nsplit=0):
        close(self.run(form, nsplit), self.want, self.backend[1], tol16=0.02, tol32=1e-4)


# heads, width, value width, latent, query latent, rotated
SIZES = {"small": (5, 24, 40, 56, 72, 12), "ragged": (3, 13, 7, 21, 19, 6), "one": (1, 32, 32, 64, 48, 16), "heads": (18, 16, 16, 130, 32, 4),
         "wide": (2, 128, 128, 192, 64, 64), "row": (3, 40, 24, 512, 32, 64), "most": (2, 24, 16, 900, 32, 16)}


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", list(SIZES))
@pytest.mark.parametrize("window", [1, 19, 64, NO_WINDOW])
def test_decode_in_a_window(backend, name, window):
    """One query per sequence, histories shorter and longer than the window, ends at and beside page and tile borders."""
    scene = Scene(backend, arch_of(*SIZES[name], window), 16, [1, 2, 18, 19, 20, 63, 64, 65, 150], [1] * 9)
    scene.check("rows")
    if backend[0] != "cpu":
        scene.check("slabs")
        for n in (1, 3, 40):
            scene.check("rows", n)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", list(SIZES))
@pytest.mark.parametrize("window", [1, 33, 70, NO_WINDOW])
def test_portions_in_a_window(backend, name, window):
    """Whole prompts, portions behind a history, single tokens among them."""
    m = arch_of(*SIZES[name], window)
    scene = Scene(backend, m, 16, [40, 1, 100, 150, 65, 141], [40, 1, 2, 70, 1, 129])
    scene.check("rows")
    if backend[0] != "cpu":
        scene.check("rows", 3)
    if backend[1] == torch.bfloat16 and m.dq <= 192 and m.dv <= 128:
        scene.check("expanded")


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("decode", [True, False])
@pytest.mark.parametrize("window", [20, 64, 129])
def test_keys_at_the_windows_edge(backend, decode, window):
    """The key just inside the window rules the result, the one just outside has no part in it; at every place of a page."""
    m = arch_of(3, 24, 24, 40, 16, 8, window)
    for n in (window + 3, window + 16, 2 * window + 7, 200):
        for edge in (window - 1, window):
            new = [1 if decode else min(n, 37), 1 if decode else 2]
            scene = Scene(backend, m, 16, [n, n - 1], new, {0: n - 1 - edge, 1: n - 2 - edge})
            for form in ("rows",) + (("expanded",) if backend[1] == torch.bfloat16 and not decode else ()):
                scene.check(form)
            loud = Scene(backend, m, 16, [n], [1], {0: n - 1 - (window - 1)})
            assert float((loud.want - Scene(backend, m, 16, [n], [1]).want).abs().max()) > 0.3 * float(loud.want.abs().max())


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("page", [8, 32, 64, 256])
def test_one_key_among_hundreds(backend, page):
    """A key far back that one query asks for, with pages of several sizes."""
    m = arch_of(4, 32, 32, 64, 16, 16, 400)
    for lookup in (0, 7, 63, 64, 255, 256, 398):
        new = [1, 130] if backend[1] == torch.bfloat16 else [1, 20]
        scene = Scene(backend, m, page, [400, 399], new, {0: lookup, 1: lookup})
        scene.check("rows")
        if backend[1] == torch.bfloat16:
            scene.check("expanded")


def test_expand_plan():
    plan = lat.ExpandPlan.make([(4, 70), (0, 0), (30, 30), (1, 33)], 20, 16, 6, "cpu")
    assert plan.first.tolist() == [2, 0, 0, 0] and plan.base.tolist() == [0, 3, 3, 5, 8] and plan.pages == 8 and plan.max_pages == 3
    assert plan.table.tolist() == [[-1, -1, 0, 1, 2, -1], [-1] * 6, [3, 4, -1, -1, -1, -1], [5, 6, 7, -1, -1, -1]]


# ---------------------------------------------------------------------------------------- short convolution
class Conv:
    def __init__(self, backend, width, taps, slots=5, carry=32):
        device, dtype = backend
        self.backend, self.width, self.W = backend, width, up(width)
        self.plain = rand(width, taps, seed=3)
        self.weight = torch.zeros(taps, self.W, dtype=dtype, device=device)
        self.weight[:, :width] = self.plain.t().to(device, dtype)
        self.spec = rec.ConvSpec(taps, self.W, carry)
        self.cache = rec.StateCache([8, carry + (taps - 1) * self.W + 4], slots, device)
        for i in range(2):
            self.cache.layer(i).fill_(1e4)      # what an earlier owner left behind

    def want(self, x):
        return x.double() + oracle.short_conv(x.double(), self.plain.double())

    def step(self, parts, decode=False):
        """parts: (rows, slot, tokens before).  A decode step runs inside the kernel that normalises the rows."""
        device, dtype = self.backend
        x = torch.nn.functional.pad(torch.cat([p[0] for p in parts]), (0, self.W - self.width)).to(device)
        lens = [p[0].shape[0] for p in parts]
        cu = None if decode else torch.tensor([0] + lens).cumsum(0).to(torch.int32).to(device)
        view = rec.StateView(self.cache, 1, torch.tensor([p[1] for p in parts], dtype=torch.int32).to(device),
                             torch.tensor([n + p[2] for n, p in zip(lens, parts)], dtype=torch.int32).to(device), cu)
        if decode:      # rows whose mean square is one are what their norm makes of them
            norm, stream = torch.empty(len(parts), self.W, dtype=dtype, device=device), x.clone().float()
            lat.stream_update(stream, self.width, 0.0, keep=True, norm_out=norm, conv=rec.ConvStep(self.weight, self.spec, view))
            y = norm
        else:
            y = rec.short_conv(x.to(dtype), self.weight, self.spec, view, max_len=max(lens))
        status(device)
        assert bool((y[:, self.width:] == 0).all())
        return y[:, :self.width].float().cpu()

    def rows(self, n, seed):
        """Signs: every row's mean square is one."""
        return torch.where(rand(n, self.width, seed=seed) > 0, 1.0, -1.0)

    def near(self, got, want):
        close(got, want, self.backend[1], tol16=0.01)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("width,taps", [(96, 4), (75, 1), (64, 2), (130, 3), (1100, 5), (48, 8), (40, 16)])
def test_convolution_in_portions(backend, width, taps):
    """Cut anywhere, shorter than the taps, of odd and even length; single tokens by both forms."""
    c = Conv(backend, width, taps)
    x = c.rows(75, 4)
    for slot, sizes in enumerate(([75], [2], [3, 1], [16, 17, 1], [1])):
        at, i, got = 0, 0, []
        while at < 75:
            n = min(sizes[i % len(sizes)], 75 - at)
            got.append(c.step([(x[at:at + n], slot, at)], decode=n == 1 and i % 3 > 0))
            at, i = at + n, i + 1
        c.near(torch.cat(got), c.want(x))
    assert bool((c.cache.layer(0) == 1e4).all()) and bool((c.cache.layer(1)[:, :, :32] == 1e4).all())


@pytest.mark.parametrize("backend", BACKENDS)
def test_convolution_of_batches(backend):
    """Unequal sequences in one step, slots handed on, rows without a slot, a step that is run again."""
    c = Conv(backend, 80, 4)
    xs = [c.rows(n, 20 + n) for n in (50, 3, 17, 33)]
    y = c.step([(xs[0], 0, 0), (xs[1], 1, 0), (xs[2], -1, 0), (xs[3][:32], 3, 0)])
    want = [c.want(x) for x in xs]
    c.near(y[:53], torch.cat(want[:2]))
    c.near(y[70:], want[3][:32])
    again = c.rows(4, 9)
    before = c.cache.layer(1).clone()
    c.step([(again[:1], 3, 32), (again[1:2], -1, 0), (again[2:3], 0, 50)], decode=True)     # ran ahead, discarded
    got = c.step([(xs[3][32:], 3, 32), (again[3:], 1, 0)], decode=True)
    c.near(got, torch.cat([want[3][32:], c.want(again[3:])]))
    assert torch.equal(before[4], c.cache.layer(1)[4]) and torch.equal(before[3, 0], c.cache.layer(1)[3, 0])


# --------------------------------------------------------------------------------------------- forget rule
FORGET = {"small": (3, 24, 40), "ragged": (5, 13, 19), "tile": (2, 64, 64), "tall": (2, 200, 16), "flat": (1, 16, 232), "two-tiles": (3, 72, 33),
          "whole": (2, 128, 128), "widest": (1, 256, 256), "many": (9, 16, 48)}


class Forget:
    def __init__(self, name, backend, slots=5, slow=False):
        self.H, self.d, self.e = FORGET[name]
        self.backend = backend
        device, dtype = backend
        self.spec = s = rec.ForgetSpec(self.H, self.d, self.e, EPS)
        C = self.H * self.d
        self.plain = {"f.b": (torch.full((C,), 7.0) if slow else rand(C, seed=1, scale=2.0)), "norm": 1 + 0.2 * rand(self.e, seed=2),
                      "lower": torch.linspace(0.0, 0.98, C) if not slow else torch.zeros(C)}
        self.plain = {k: v.to(torch.bfloat16).float() for k, v in self.plain.items()}
        w = rec.ForgetWeights(torch.zeros(s.gate_col, dtype=dtype, device=device), torch.ones(s.gate_col, dtype=dtype, device=device),
                              torch.zeros(s.m, dtype=dtype, device=device))
        w.bias.view(self.H, s.n)[:, :self.d] = self.plain["f.b"].view(self.H, -1).to(device, dtype)
        w.lower.view(self.H, s.n)[:, :self.d] = self.plain["lower"].view(self.H, -1).to(device, dtype)
        w.norm[:self.e] = self.plain["norm"].to(device, dtype)
        self.w = w
        self.cache = rec.StateCache([8, s.carry + 12], slots, device)
        for i in range(2):
            self.cache.layer(i).fill_(1e4)

    def rows(self, T, seed):
        """(queries, gates, values) before their activations"""
        return rand(T, self.H, self.d, seed=seed), rand(T, self.H, self.d, seed=seed + 1, scale=2.0), rand(T, self.H, self.e, seed=seed + 2)

    def want(self, x):
        q, z, v = (t.double() for t in x)
        f = oracle.forget(z.flatten(1) + self.plain["f.b"].double(), self.plain["lower"].double()).view_as(z)
        o, _ = oracle.recurrence(oracle.silu(q), f, v)
        return (oracle.rms(o, EPS) * self.plain["norm"].double()).flatten(1)

    def step(self, parts, decode=False, source="slabs"):
        """parts: (rows, slot, tokens before)"""
        device, dtype = self.backend
        s, lens = self.spec, [p[0][0].shape[0] for p in parts]
        T = sum(lens)
        y = torch.zeros(T, s.proj_cols)
        for first, n, k, i in ((0, s.n, self.d, 0), (s.gate_col, s.n, self.d, 1), (s.value_col, s.m, self.e, 2)):
            y[:, first:first + self.H * n].view(T, self.H, n)[..., :k] = torch.cat([p[0][i] for p in parts])
        cu = None if decode else torch.tensor([0] + lens).cumsum(0).to(torch.int32).to(device)
        view = rec.StateView(self.cache, 1, torch.tensor([p[1] for p in parts], dtype=torch.int32).to(device),
                             torch.tensor([n + p[2] for n, p in zip(lens, parts)], dtype=torch.int32).to(device), cu)
        got = rec.forget_mix(as_branch(y, source, self.backend), s, self.w, view)
        status(device)
        got = got.float().cpu().view(T, self.H, s.m)
        assert bool((got[..., self.e:] == 0).all())
        return got[..., :self.e].flatten(1)

    def near(self, got, want, tol16=0.015):
        close(got, want, self.backend[1], tol16=tol16, tol32=1e-4)


def cut(x, lo, hi):
    return tuple(t[lo:hi] for t in x)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", list(FORGET))
def test_forget_rule_over_a_sequence(backend, name):
    m = Forget(name, backend)
    for T in (1, 2, 15, 16, 17, 33, 90):
        x = m.rows(T, 100 + T)
        for source in ("slabs", "rows"):
            m.near(m.step([(x, 3, 0)], source=source), m.want(x))


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", list(FORGET))
def test_forget_rule_token_by_token(backend, name):
    m = Forget(name, backend)
    x = m.rows(40, 3)
    m.near(torch.cat([m.step([(cut(x, i, i + 1), 1, i)], decode=True, source="rows" if i % 5 == 2 else "slabs") for i in range(40)]), m.want(x))


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("sizes", [[2], [3], [1, 2], [16, 4], [17, 15], [33, 1, 1], [5, 40]])
def test_forget_rule_in_portions(backend, sizes):
    """Portions of odd and even length, so that a version is read and written by the same step."""
    m = Forget("ragged", backend)
    x, at, i, got = m.rows(75, 4), 0, 0, []
    while at < 75:
        n = min(sizes[i % len(sizes)], 75 - at)
        got.append(m.step([(cut(x, at, at + n), 2, at)], decode=n == 1 and i % 2 == 1 and at > 0))
        at, i = at + n, i + 1
    m.near(torch.cat(got), m.want(x))


@pytest.mark.parametrize("backend", BACKENDS)
def test_forget_rule_in_batches(backend):
    """Portions beside single tokens, slots handed on, a repeated step, rows without a slot."""
    m = Forget("two-tiles", backend)
    xs = [m.rows(n, 50 + n) for n in (61, 30, 45, 20)]
    out, at = [[] for _ in xs], [0] * 4
    for step in ([(0, 30), (1, 2)], [(0, 1), (1, 15), (2, 40)], [(2, 2), (0, 1)], [(1, 13), (0, 29), (2, 3)]):
        y, base = m.step([(cut(xs[r], at[r], at[r] + n), r, at[r]) for r, n in step]), 0
        for r, n in step:
            out[r].append(y[base:base + n])
            base, at[r] = base + n, at[r] + n
    for r in range(3):
        m.near(torch.cat(out[r]), m.want(xs[r]))
    m.near(m.step([(cut(xs[3], 0, 19), 1, 0)]), m.want(xs[3])[:19])            # slot 1 once more
    other = m.rows(3, 7)
    before = m.cache.layer(1).clone()
    y = m.step([(cut(other, 0, 1), 1, 19), (cut(other, 1, 2), -1, 0), (cut(other, 2, 3), 4, 0)], decode=True)   # ran ahead, discarded
    assert bool((y[1] == 0).all())
    m.near(m.step([(cut(xs[3], 19, 20), 1, 19)], decode=True), m.want(xs[3])[19:])
    y = m.step([(other, -1, 4)])
    assert bool((y == 0).all()) and torch.equal(m.cache.layer(1)[:1], before[:1]) and bool((m.cache.layer(0) == 1e4).all())
    assert bool((m.cache.layer(1)[:, :, m.spec.carry:] == 1e4).all())


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("decode", [False, True])
def test_a_far_write_is_remembered(backend, decode):
    """Gates that are all but open, and one token that writes much: it rules hundreds of tokens later, and not before."""
    m = Forget("tile", backend, slow=True)
    q, z, v = m.rows(401, 12)
    z = 0.2 * z
    z[20], v = -14.0, 0.3 * v
    v[20] = 30.0 * torch.sign(v[20])
    x = (q.abs() + 1.0, z, v)
    want = m.want(x)
    if decode:
        got = torch.cat([m.step([(cut(x, 0, 300), 0, 0)])] + [m.step([(cut(x, i, i + 1), 0, i)], decode=True) for i in range(300, 401)])
    else:
        got = torch.cat([m.step([(cut(x, 0, 200), 0, 0)], source="rows"), m.step([(cut(x, 200, 401), 0, 200)])])
    m.near(got, want, tol16=0.03)
    v2 = v.clone()
    v2[20] = v[21]
    assert float((m.want((x[0], z, v2))[400] - want[400]).abs().max()) > 0.2 * float(want[400].abs().max())


# ------------------------------------------------------------------------------------------- depth average
@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("width,T", [(64, 3), (75, 5), (1200, 2), (4100, 3), (352, 300), (2048, 260)])
def test_depth_average(backend, width, T):
    """Results are kept in 32-bit and summed with their weights; the norm, the copy and the stream see the sum."""
    device, dtype = backend
    W, vocab, mult = up(width), 11, 0.7
    wide = lambda t: torch.nn.functional.pad(t, (0, W - width))  # noqa: E731
    table, ids = wide(rand(vocab, width, seed=1)), torch.arange(T) % vocab
    x, history = torch.full((T, W), 7.0, device=device), torch.full((5, T, W), 1e4, device=device)
    norm, raw, w = torch.empty(T, W, dtype=dtype, device=device), torch.empty(T, W, dtype=dtype, device=device), wide(rand(width, seed=2))
    kw = dict(norm_weight=w.to(device, dtype), norm_out=norm, raw_out=raw, history=history)
    lat.stream_update(x, width, EPS, keep=False, ids=ids.to(device), table=table.to(device, dtype), embed_mult=3.0, depth=0, **kw)
    rows, now = [3.0 * table[ids].double()], 3.0 * table[ids].double()
    close(x, now, torch.float32, tol32=1e-6)
    for i in range(4):
        y, a = wide(rand(2, T, width, seed=10 + i)), rand(i + 2, seed=20 + i)
        lat.stream_update(x, width, EPS, keep=True, a=Branch(slabs=y.to(device)), mult=mult, depth=i + 1, depth_weight=a.to(device), **kw)
        rows.append(now + mult * y.double().sum(0))
        close(history[i + 1], rows[-1], torch.float32, tol32=3e-6)
        now = oracle.depth_average(rows, a.double())
        close(x, now, torch.float32, tol32=3e-6)
        close(raw, now, dtype)
        close(norm[:, :width], oracle.rms(now[:, :width], EPS) * w[:width].double(), dtype)
    status(device)


# ------------------------------------------------------------------------------- routing and bounded experts
# outputs, chosen, groups, kept, scale
ROUTES = {"groups": (15, 4, 5, 3, 2.2), "single": (6, 2, 6, 3, 0.7), "one-group": (5, 4, 1, 1, 1.0), "many": (96, 6, 8, 3, 2.5), "wide": (260, 8, 13, 4, 1.5), "all": (4, 4, 2, 2, 1.0)}


def routing(T, name, device, seed=7):
    E, top, groups, keep, scale = ROUTES[name]
    z, a = rand(T, E, seed=seed, scale=2.0) + 1e-3 * torch.randn(T, E, generator=torch.Generator().manual_seed(seed + 5)), rand(T, E, seed=seed + 1)
    s = moe.Scored(torch.zeros(E, device=device), 0, groups, keep, scale, sigmoid=True, group_best=2)
    chosen = [dict(oracle.route(z[t].double(), {"top": top, "scale": scale, "groups": {"count": groups, "keep": keep}})) for t in range(T)]
    return Branch(slabs=torch.stack([a, z - a]).to(device)), s, chosen, E, top


@pytest.mark.parametrize("backend", BACKENDS[:2])
@pytest.mark.parametrize("name", list(ROUTES))
@pytest.mark.parametrize("T", [1, 9, 128, 129, 400])
def test_sigmoid_routing(backend, name, T):
    device, _ = backend
    b, s, chosen, E, top = routing(T, name, device)
    slots = torch.arange(T)
    slots[T // 2] = -1 if T > 1 else 0
    r = moe.route(b, top, E, 0, slots.to(device), scored=s)
    pos, weight, table = r.pos.cpu(), r.weight.cpu(), r.groups.cpu()[:int(r.n_groups[0])].tolist()
    expert = {row: e for e, first, n, _ in table for row in range(first, first + n)}
    for t in range(T):
        if slots[t] < 0:
            assert bool((pos[t] < 0).all()) and bool((weight[t] == 0).all())
            continue
        got = {expert[int(p)]: float(w) for p, w in zip(pos[t], weight[t])}
        assert got.keys() == chosen[t].keys() and all(abs(got[e] - chosen[t][e]) < 1e-5 for e in got), t
    status(device)


@pytest.mark.parametrize("backend", BACKENDS[:2])
def test_two_good_outputs_beat_one_very_good(backend):
    """A group counts by the sum of its two best; equal scores go to the lowest."""
    device, _ = backend
    z = torch.tensor([[4.0, -9.0, -9.0, 1.0, 1.0, -9.0, 0.9, 0.9, 0.9], [0.0] * 9])
    s = moe.Scored(torch.zeros(9, device=device), 0, 3, 1, 1.0, sigmoid=True, group_best=2)
    r = moe.route(Branch(slabs=z[None].to(device)), 2, 9, 0, torch.arange(2).to(device), scored=s)
    table = r.groups.cpu()[:int(r.n_groups[0])].tolist()
    assert [(e, n) for e, _, n, _ in table] == [(0, 1), (1, 1), (3, 1), (4, 1)]
    assert torch.allclose(r.weight.cpu()[0], torch.sigmoid(torch.ones(2)), atol=1e-6) and torch.allclose(r.weight.cpu()[1], torch.full((2,), 0.5))


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("T", [1, 5, 128, 140, 500])
@pytest.mark.parametrize("name,W,F", [("groups", 96, 48), ("single", 112, 208), ("one-group", 336, 144)])
def test_bounded_experts(backend, T, name, W, F):
    """Gates and inputs on both sides of the bound."""
    device, dtype = backend
    b, s, chosen, E, top = routing(T, name, device, seed=31)
    limit, x = 1.25, rand(T, W, seed=3)
    gu, down = rand(E, 2 * F, W, seed=4, scale=2 * W ** -0.5), rand(E, W, F, seed=5, scale=F ** -0.5)
    r = moe.route(b, top, E, 0, torch.arange(T).to(device), f32=dtype == torch.float32, scored=s)
    got = moe.expert_ffn(x.to(device, dtype), r, gu.to(device, dtype), down.to(device, dtype), "bounded", limit)
    want = torch.zeros(T, W, dtype=torch.float64)
    for t in range(T):
        for e, weight in chosen[t].items():
            h = x[t].double() @ gu[e].double().T
            want[t] += weight * (oracle.bounded_glu(h[:F], h[F:], limit) @ down[e].double().T)
    stream = torch.zeros((T, W), device=device)
    lat.stream_update(stream, W, 1e-5, keep=False, a=got, raw_out=torch.empty((T, W), dtype=dtype, device=device))
    close(stream, want, dtype, tol16=0.015)
    status(device)


@pytest.mark.parametrize("backend", [GPU16])
def test_unit_far_past_its_bounds(backend):
    """Gates of minus a thousand give nothing, gates and inputs of a thousand what the bound gives."""
    device, dtype = backend
    W = F = 64
    x = torch.ones(3, W)
    gate, upw = torch.zeros(F, W), torch.zeros(F, W)
    gate[:, 0], upw[:, 0] = torch.where(torch.arange(F) % 2 == 0, 1000.0, -1000.0), torch.where(torch.arange(F) % 4 < 2, 1000.0, -1000.0)
    s = moe.Scored(torch.zeros(1, device=device), sigmoid=True, group_best=2)
    r = moe.route(Branch(slabs=torch.zeros(1, 3, 1, device=device)), 1, 1, 0, torch.arange(3).to(device), scored=s)
    got = moe.expert_ffn(x.to(device, dtype), r, torch.cat([gate, upw])[None].to(device, dtype), torch.eye(W)[None].to(device, dtype), "bounded", 3.0).value()
    want = 0.5 * oracle.bounded_glu(gate[:, 0].double(), upw[:, 0].double(), 3.0)
    close(got, want.expand(3, -1), dtype)
