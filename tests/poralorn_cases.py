"""Small Poralorn configurations and weights for the tests."""

import torch

from prism_infer_b200.models.architecture import PoralornArch
from prism_infer_b200.models.weights import random_weights
from replay_helpers import checkpoint, engine, error, portions, replay, tokens  # noqa: F401


def mixer(heads, dim, vdim, kv_rank, scale):
    return {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale}


def config(layers, *, vocab=200, width=96, loop=None, eps=1e-5, mult=0.5, cap=10.0):
    """``layers``: (mixer dictionary, feed-forward width or 0) per layer."""
    out = {"architecture": "Poralorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
           "logit_softcap": cap,
           "layers": [{"type": "latent_attention", "mixer": m, "mlp": {"kind": "dense", "ff": f} if f else None} for m, f in layers]}
    if loop is not None:
        out["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return out


CASES = {
    # every size different, value width below and above the key width, odd head counts, ranks that fill no tile
    "uneven": config([(mixer(3, 40, 24, 72, 0.21), 136), (mixer(5, 16, 48, 40, 0.3), 0), (mixer(2, 24, 24, 130, 0.17), 56)],
                     vocab=211, width=120, loop=(1, 3, 2), eps=3e-4, mult=0.7, cap=9.0),
    # nothing is a multiple of eight
    "ragged": config([(mixer(3, 13, 7, 21, 0.4), 37), (mixer(1, 30, 19, 67, 0.15), 51)], vocab=97, width=75, loop=(0, 1, 3), cap=6.0),
    # the loop covers every layer and runs once
    "once": config([(mixer(4, 32, 32, 64, 0.18), 96)], vocab=160, width=64, loop=(0, 1, 1), mult=1.0),
    # the loop is the last layer
    "tail": config([(mixer(4, 72, 72, 136, 0.12), 160), (mixer(4, 72, 72, 136, 0.1), 160)], vocab=192, width=128, loop=(1, 2, 4), mult=0.25,
                   cap=20.0),
    # no loop, wide heads (no square tensor-core path), wide latent
    "wide": config([(mixer(2, 160, 96, 320, 0.08), 64), (mixer(9, 48, 48, 600, 0.14), 0)], vocab=128, width=112),
}


def make(name, seed=0):
    """(config, architecture, float32 weights holding bf16 values).  Gains and step vectors are spread out so that
    a swapped or missing one shows."""
    cfg = CASES[name]
    arch = PoralornArch.from_hf_config(cfg)
    w = random_weights(arch, seed=seed)
    g = torch.Generator().manual_seed(seed + 17)
    for k in w:
        if arch.init_kind(k) == "norm":
            w[k] = 0.6 + 0.8 * torch.rand(w[k].shape, generator=g)
        elif arch.init_kind(k) == "bias":
            w[k] = 0.5 * torch.randn(w[k].shape, generator=g)
        elif k == "embed":
            w[k] = torch.randn(w[k].shape, generator=g)
        w[k] = w[k].to(torch.bfloat16).float()
    w["head"] = (w["head"] * 4).to(torch.bfloat16).float()
    return cfg, arch, w
