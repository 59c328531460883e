"""Backends, operands and comparison of the op tests."""

import pytest
import torch

CPU = pytest.param(("cpu", torch.float32), id="cpu")
GPU32 = pytest.param(("cuda:0", torch.float32), marks=pytest.mark.gpu, id="gpu-float32")
GPU16 = pytest.param(("cuda:0", torch.bfloat16), marks=pytest.mark.gpu, id="gpu-bfloat16")
BACKENDS = [CPU, GPU32, GPU16]


def rand(*shape, seed=0, scale=1.0, dtype=torch.float32, device="cpu"):
    """Values every type can hold: drawn on the CPU and rounded to bf16."""
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(torch.bfloat16).to(dtype).to(device)


def close(got, want, dtype, tol16=0.012, tol32=2e-5):
    got, want = got.detach().double().cpu(), want.double()
    assert got.shape == want.shape
    err = (got - want).abs().max() / want.abs().max().clamp_min(1e-6)
    assert float(err) < (tol16 if dtype == torch.bfloat16 else tol32), float(err)
