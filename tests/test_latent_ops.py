"""Ops of the latent-attention family, each against a plain float64 statement: stacked projections, the 32-bit
residual stream, latent attention in its absorbed and expanded forms.  CPU statements, and the kernels on a B200."""

import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import poralorn_oracle as oracle  # noqa: E402
from op_helpers import BACKENDS, close, rand  # noqa: E402

from prism_infer_b200 import ops  # noqa: E402
from prism_infer_b200.ops import latent as lat  # noqa: E402

# ------------------------------------------------------------------------------------------ projections
@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("tokens", [1, 7, 40, 130, 530])
def test_stacked_projection(backend, tokens):
    """Every activation with its own scale and bias, at token counts that take every tile form."""
    device, dtype = backend
    K = 136
    parts = [(48, 0.7, None), (176, -1.3, "gelu"), (16, 2.0, "sigmoid"), (80, 0.5, "gelu_tanh"), (32, 1.0, None)]
    M = sum(p[0] for p in parts)
    x, w, b = rand(tokens, K, seed=1), rand(M, K, seed=2, scale=K ** -0.5), rand(M, seed=3)
    z = x.double() @ w.double().T
    want, at = [], 0
    for rows, alpha, act in parts:
        y = alpha * z[:, at:at + rows] + b[at:at + rows].double()
        if act == "gelu":
            y = oracle.gelu_exact(y)
        elif act == "sigmoid":
            y = oracle.sigmoid(y)
        elif act == "gelu_tanh":
            y = 0.5 * y * (1 + torch.tanh((2 / torch.pi) ** 0.5 * (y + 0.044715 * y ** 3)))
        want.append(y)
        at += rows
    got = lat.linear_sections(x.to(device, dtype), w.to(device, dtype), lat.Sections(parts), bias=b.to(device, dtype))
    close(got, torch.cat(want, 1), dtype)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("rows,vocab", [(1, 97), (5, 1000), (70, 515), (600, 97)])
def test_capped_logits(backend, rows, vocab):
    device, dtype = backend
    x, w = rand(rows, 72, seed=1), rand(vocab, 72, seed=2)
    want = oracle.softcap(0.9 * (x.double() @ w.double().T), 11.0)
    assert float(want.abs().max()) > 10.0  # the cap is at work
    got = lat.linear_sections(x.to(device, dtype), w.to(device, dtype), lat.Sections([(vocab, 0.9, "softcap")], 11.0), out_f32=True)
    assert got.dtype == torch.float32
    close(got, want, dtype, tol16=2e-5)


def test_sections_are_checked():
    with pytest.raises(KeyError):
        lat.Sections([(16, 1.0, "relu")])
    with pytest.raises(AssertionError):
        lat.linear_sections(rand(2, 8), rand(32, 8), lat.Sections([(16, 1.0, None)]))


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("tokens", [3, 300, 700])
def test_slabs(backend, tokens):
    device, dtype = backend
    x, w = rand(tokens, 640, seed=1), rand(96, 640, seed=2, scale=0.05)
    got = lat.linear_slabs(x.to(device, dtype), w.to(device, dtype))
    assert got.dtype == torch.float32
    close(got.sum(0), x.double() @ w.double().T, dtype, tol16=2e-5)


# ----------------------------------------------------------------------------------------- residual stream
@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("width,padded", [(64, 64), (75, 80), (1200, 1200), (4100, 4112)])
def test_stream_update(backend, width, padded):
    device, dtype = backend
    T, vocab, eps, mult = 5, 23, 3e-3, 0.37
    pad = padded - width

    def padded_rows(t):
        return torch.nn.functional.pad(t, (0, pad))

    table, ids = padded_rows(rand(vocab, width, seed=1)), torch.tensor([3, 0, 22, 3, 7])
    x = torch.full((T, padded), 7.0, device=device)
    norm = torch.full((T, padded), 9.0, dtype=dtype, device=device)
    pair = torch.zeros((T, 2 * padded), dtype=dtype, device=device)
    lat.stream_update(x, width, eps, keep=False, ids=ids.to(device), table=table.to(device, dtype), norm_out=norm,
                      raw_out=pair[:, :padded], embed_out=pair[:, padded:])
    want = table[ids].double()
    close(x, want, torch.float32, tol32=1e-7)
    close(norm, padded_rows(oracle.rms(want[:, :width], eps)), dtype)
    close(pair, torch.cat([want, want], 1), dtype)
    # both branches: slabs with a gate taken from a wider buffer, rows with another gate of it
    slabs, rows = padded_rows(torch.randn(3, T, width, generator=torch.Generator().manual_seed(5))), padded_rows(rand(T, width, seed=6))
    gates = rand(T, 3 * padded, seed=7).to(device, dtype)
    ga, gb = gates[:, :padded], gates[:, padded:2 * padded]
    lat.stream_update(x, width, eps, keep=True, a=lat.Branch(slabs=slabs.to(device), gate=ga),
                      b=lat.Branch(rows=rows.to(device, dtype), gate=gb), mult=mult, norm_out=norm)
    want = want + mult * (slabs.double().sum(0) * ga.double().cpu() + rows.double() * gb.double().cpu())
    close(x, want, torch.float32, tol32=2e-6)
    close(norm, padded_rows(oracle.rms(want[:, :width], eps)), dtype)
    # one branch, no gate, a bias vector, replacing the stream
    bias = padded_rows(rand(1, width, seed=8))[0]
    lat.stream_update(x, width, eps, keep=False, a=lat.Branch(slabs=slabs.to(device)), bias=bias.to(device, dtype), norm_out=norm)
    close(x, slabs.double().sum(0) + bias.double(), torch.float32, tol32=2e-6)


@pytest.mark.parametrize("backend", BACKENDS)
def test_stream_keeps_what_sixteen_bits_would_lose(backend):
    """A thousand additions far below a bf16 step of the stream arrive."""
    device, dtype = backend
    x = torch.full((2, 64), 256.0, device=device)
    small = torch.full((1, 2, 64), 2.0 ** -7, device=device)
    norm = torch.empty((2, 64), dtype=dtype, device=device)
    for _ in range(1024):
        lat.stream_update(x, 64, 1e-5, keep=True, a=lat.Branch(slabs=small), norm_out=norm)
    assert torch.equal(x.cpu(), torch.full((2, 64), 264.0))


# ---------------------------------------------------------------------------------------- latent attention
def up(n, to):
    return -(-n // to) * to


class Scene:
    """Sequences whose histories are in a paged cache and whose new tokens are in hand, with the plain result.

    ``lookups``: sequence -> key position its last new token is made to look at (its query is that key, scaled, so the
    score stands out among all others)."""

    def __init__(self, backend, heads, dim, vdim, rank, page, hist, new, lookups=None, spare=3, seed=0):
        self.backend, self.page = backend, page
        device, dtype = backend
        self.hist, self.new, self.eps, scale = hist, new, 2e-4, dim ** -0.5
        Rc = up(rank, 64)
        dq, dv = up(dim, 8), up(vdim, 8)
        if max(dq, dv) <= 128:
            dq = dv = max(dq, dv)
        weight, uk, uv = 1 + 0.3 * rand(rank, seed=seed + 1), rand(heads * dim, rank, seed=seed + 2, scale=rank ** -0.5), \
            rand(heads * vdim, rank, seed=seed + 3, scale=rank ** -0.5)
        weight = weight.to(torch.bfloat16).float()
        ukv = torch.zeros(heads * (dq + dv), Rc)
        ukv[:heads * dq].view(heads, dq, Rc)[:, :dim, :rank] = uk.view(heads, dim, rank)
        ukv[heads * dq:].view(heads, dv, Rc)[:, :vdim, :rank] = uv.view(heads, vdim, rank)
        self.lw = lat.LatentWeights(heads, dq, dv, rank, scale, weight.to(device, dtype), ukv.to(device, dtype))
        total = [h + n for h, n in zip(hist, new)]
        pages = [up(t, page) // page for t in total]
        self.cache = ops.KVCache(2, sum(pages) + spare, 1, page, Rc, ops.KV_BF16, device, dtype=dtype, planes=1)
        self.cache.payload.copy_(rand(*self.cache.payload.shape, seed=seed + 4, scale=30.0))  # what earlier users left behind
        order = torch.randperm(sum(pages) + spare, generator=torch.Generator().manual_seed(seed)).tolist()
        table = torch.full((len(total), max(pages) + 1), -1, dtype=torch.int32)
        for s, n in enumerate(pages):
            for i in range(n):
                table[s, i] = order.pop()
        self.table = table.to(device)
        raws, qs, gates, outs, self.slots, first = [], [], [], [], [], []
        for s, (h, n) in enumerate(zip(hist, new)):
            raw = rand(h + n, rank, seed=seed + 10 + s)
            c = oracle.rms(raw.double(), self.eps) * weight.double()
            if dtype == torch.bfloat16:
                c = c.to(torch.bfloat16).double()
            k, v = (c @ uk.double().T).view(-1, heads, dim), (c @ uv.double().T).view(-1, heads, vdim)
            q = rand(n, heads, dim, seed=seed + 20 + s)
            if lookups and s in lookups:
                target = k[lookups[s]]
                q[-1] = (target / target.norm(dim=-1, keepdim=True) * 25.0 / scale / target.norm(dim=-1, keepdim=True)).to(torch.bfloat16)
            gate = oracle.sigmoid(rand(n, heads * vdim, seed=seed + 30 + s).double()).to(torch.bfloat16)
            full_q = torch.cat([torch.zeros(h, heads, dim), q]).double()
            o = oracle.causal_softmax_attention(full_q, k, v, scale)[h:].reshape(n, -1) * gate.double()
            pos = torch.arange(h + n)
            slot = table[s, pos // page].long() * page + pos % page
            raws.append(raw), qs.append(q), gates.append(gate), outs.append(o)
            self.slots.append(slot)
            if h:  # the history, through the op itself
                lat.latent_norm_store(raw[:h].to(device, dtype), self.lw, self.eps, slot[:h].to(device), self.cache, 1)
        T = sum(new)

        def pad_heads(t, real, padded):
            z = torch.zeros(T, heads, padded)
            z[..., :real] = t.reshape(T, heads, real)
            return z.reshape(T, heads * padded)

        # the three inputs sit side by side in one wide row, as a stacked projection leaves them
        q, raw, gate = pad_heads(torch.cat(qs), dim, dq), torch.cat([r[h:] for r, h in zip(raws, hist)]), pad_heads(torch.cat(gates), vdim, dv)
        cols = [0, up(heads * dq, 16), up(heads * dq, 16) + up(rank, 16)]
        wide = torch.full((T, cols[2] + up(heads * dv, 16)), 5.0)
        for at, t in zip(cols, (q, raw, gate)):
            wide[:, at:at + t.shape[1]] = t
        wide = wide.to(device, dtype)
        self.q, self.raw, self.gate = (wide[:, at:at + t.shape[1]] for at, t in zip(cols, (q, raw, gate)))
        self.want = pad_heads(torch.cat(outs).float(), vdim, dv)
        self.new_slots = torch.cat([sl[h:] for sl, h in zip(self.slots, hist)]).to(device)
        self.kv_lens = torch.tensor(total, dtype=torch.int32, device=device)
        self.cu_q = torch.tensor([0] + torch.tensor(new).cumsum(0).tolist(), dtype=torch.int32, device=device)
        self.cu_kv = torch.tensor([0] + torch.tensor(total).cumsum(0).tolist(), dtype=torch.int32, device=device)
        self.total = total

    def absorbed(self, nsplit=0):
        cu = None if all(n == 1 for n in self.new) else self.cu_q
        return lat.latent_attention_absorbed(self.q, self.raw, self.gate, self.lw, self.eps, self.new_slots, self.cache, 1, self.table,
                                             self.kv_lens, cu_seqlens_q=cu, max_q_len=max(self.new), nsplit=nsplit)

    def expanded(self):
        return lat.latent_attention_expanded(self.q, self.raw, self.gate, self.lw, self.eps, self.new_slots, self.cache, 1, self.table,
                                             self.cu_q, max(self.new), cu_seqlens_kv=self.cu_kv if any(self.hist) else None,
                                             total_kv=sum(self.total), max_kv_len=max(self.total))

    def forms(self):
        device, dtype = self.backend
        yield "absorbed", self.absorbed()
        if dtype == torch.bfloat16:
            for n in (1, 2, 7, 33, 64):
                yield f"absorbed, {n} splits", self.absorbed(n)
            if self.lw.dq == self.lw.dv and self.lw.dq <= 128:
                yield "expanded", self.expanded()

    def check(self):
        for name, got in self.forms():
            err = (got.double().cpu() - self.want.double()).abs().max() / self.want.double().abs().max()
            assert float(err) < (0.025 if self.backend[1] == torch.bfloat16 else 2e-5), (name, float(err))
        if self.backend[0] != "cpu":
            from prism_infer_b200.ops import native

            native.check_status()


SIZES = {"uneven": (3, 40, 24, 72), "production": (32, 128, 128, 512), "no square heads": (2, 160, 96, 320), "widest": (1, 16, 16, 1000),
         "sixteen": (16, 64, 64, 128), "small": (5, 8, 8, 64), "odd": (7, 72, 13, 200), "padded": (17, 96, 80, 250)}


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("size", list(SIZES))
def test_prompts_without_history(backend, size):
    Scene(backend, *SIZES[size], 16, [0, 0, 0], [37, 1, 70]).check()


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("size", list(SIZES))
def test_portions_over_history(backend, size):
    Scene(backend, *SIZES[size], 16, [130, 0, 63, 5], [2, 33, 1, 17]).check()


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("size", list(SIZES))
def test_decode_steps_of_unequal_sequences(backend, size):
    Scene(backend, *SIZES[size], 64, [0, 1, 63, 64, 65, 200], [1] * 6).check()


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("page", [16, 64, 256])
def test_one_key_stands_out(backend, page):
    """Decoded tokens and portions whose query is one far key: first, last, beside every page and tile border, itself."""
    spots = [0, 1, 15, 16, 31, 32, 63, 64, 65, 127, 128, 190, 191, 255, 256, 299, 300]
    for new in (1, 3):
        hist = [301 - new] * len(spots)
        scene = Scene(backend, 4, 64, 64, 128, page, hist, [new] * len(spots), {s: p for s, p in enumerate(spots)})
        scene.check()
        last = scene.want.view(len(spots), new, -1)[:, -1]
        assert float((last[1:] - last[:-1]).abs().amax(-1).min()) > 0.1  # different keys give different rows


@pytest.mark.parametrize("backend", BACKENDS)
def test_order_of_the_batch_and_pages_do_not_matter(backend):
    """One sequence alone and among others, over other pages: the same row up to rounding."""
    alone = Scene(backend, 6, 32, 32, 64, 16, [77], [5])
    crowd = Scene(backend, 6, 32, 32, 64, 16, [77, 3, 150], [5, 40, 1], spare=9)
    a, b = alone.absorbed(), crowd.absorbed()
    close(b[:5], a.double().cpu(), backend[1], tol16=0.01, tol32=1e-5)


@pytest.mark.parametrize("backend", BACKENDS)
def test_padding_rows_of_a_decode_batch(backend):
    """Rows without a sequence (no slot, no keys, no pages) give zeros and touch nothing."""
    scene = Scene(backend, 4, 32, 32, 64, 16, [20, 33], [1, 1])
    scene.new_slots[1], scene.kv_lens[1], scene.table[1] = -1, 0, -1
    before = scene.cache.payload.clone()
    got = scene.absorbed()
    assert bool((got[1] == 0).all())
    close(got[:1], scene.want[:1].double(), scene.backend[1], tol16=0.025)
    changed = (scene.cache.payload != before).flatten(0, 3).any(-1).nonzero()
    assert len(changed) <= 1  # the one new latent


@pytest.mark.gpu
def test_bounds_are_checked_on_the_device(cuda_device):
    """A page id beyond the cache and a slot beyond it are skipped and recorded, not accessed."""
    from prism_infer_b200.ops import native

    native.read_status(reset=True)
    scene = Scene(("cuda:0", torch.bfloat16), 4, 32, 32, 64, 16, [40], [1])
    scene.table[0, 1] = 10_000
    scene.absorbed()
    assert native.read_status(reset=True)["latent"][0] == 3
    scene.table[0, 1] = -1
    scene.new_slots[0] = 10 ** 9
    scene.absorbed()
    assert native.read_status(reset=True)["latent"][0] == 3
    native.check_status()


def test_route_of_a_prompt_step():
    """Whole prompts go through explicit keys and values, decode-like steps stay absorbed, wide heads always do."""
    lw = lat.LatentWeights(32, 128, 128, 512, 0.1, torch.empty(0), torch.empty(0))
    assert lat.expanded_is_cheaper(lw, 512, 2048, 2048 * 2048)
    assert not lat.expanded_is_cheaper(lw, 512, 4096, 4096)
    assert not lat.expanded_is_cheaper(lat.LatentWeights(32, 192, 128, 512, 0.1, torch.empty(0), torch.empty(0)), 512, 2048, 2048 * 2048)
    assert not lat.expanded_is_cheaper(lw, 512, 10 ** 6, 10 ** 9)  # the explicit keys would not fit their scratch


def test_single_plane_pages_are_copied_and_counted():
    cache = ops.KVCache(3, 5, 1, 16, 64, ops.KV_BF16, "cpu", dtype=torch.float32, planes=1)
    cache.payload.copy_(rand(*cache.payload.shape))
    assert cache.bytes_per_page() == 3 * 16 * 64 * 4 and cache.n_slabs == 3
    want = cache.latent(2)[1].clone()
    ops.kv_page_copy(cache, cache, [1], [4])
    assert torch.equal(cache.latent(2)[4], want)
