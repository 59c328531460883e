"""Small Fosulix configurations and weights for the tests."""

import torch

from prism_infer_b200.models.architecture import FosulixArch
from prism_infer_b200.models.weights import random_weights
from replay_helpers import checkpoint, engine, error, portions, replay, tokens  # noqa: F401


def yarn(factor=4.0, original=64, fast=6.0, slow=1.0):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def latent(heads, dim, vdim, *, rank, q_rank, rot, window, base=700.0, scaling=None, kv_from=None):
    return {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank, "rot_dim": rot, "scale": 1.5 * (dim + rot) ** -0.5,
            "rot": {"base": base, "dims": rot, **({"scaling": scaling} if scaling else {})},
            **({"mask": {"size": window}} if window else {}), **({"kv_from": kv_from} if kv_from is not None else {})}


def forget(heads, dim, vdim):
    return {"heads": heads, "dim": dim, "vdim": vdim}


def moe(experts, top, ff, *, groups=None, scale=1.0, limit=1.75):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit},
            "router": {"experts": experts, "top": top, "scale": scale, **({"groups": {"count": groups[0], "keep": groups[1]}} if groups else {})}}


def config(layers, *, vocab=200, width=96, eps=1e-5, embed=2.0, taps=4, mult=0.8):
    """``layers``: (mixer dictionary, feed-forward dictionary or None) per layer."""
    return {"architecture": "Fosulix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed},
            "canon": {"taps": taps}, "residual_mult": mult,
            "layers": [{"type": "latent_attention" if "kv_rank" in m else "hgrn2", "mixer": m, "mlp": f} for m, f in layers]}


A = latent(5, 24, 40, rank=56, q_rank=72, rot=12, window=19, scaling=yarn())
B = latent(3, 13, 7, rank=21, q_rank=19, rot=6, window=33)
C = latent(4, 32, 32, rank=64, q_rank=48, rot=16, window=27, scaling=yarn(2.5, 96, 9.0, 2.0))
D = latent(2, 128, 128, rank=192, q_rank=128, rot=64, window=70, base=5000.0, scaling=yarn(8.0, 48, 4.0, 0.5))
E = latent(1, 160, 144, rank=520, q_rank=40, rot=60, window=45)
CASES = {
    # every size different, both mixers, latents of another layer behind another window, groups of experts
    "uneven": config([(forget(3, 24, 40), moe(8, 3, 48, groups=(4, 2), scale=1.7, limit=1.5)), (A, moe(9, 2, 40, groups=(3, 2), scale=0.6, limit=0.7)),
                      (A | {"mask": {"size": 8}, "heads": 2, "dim": 40, "vdim": 24, "q_rank": 40, "scale": 0.21, "kv_from": 1}, None),
                      (forget(2, 40, 16), moe(5, 4, 33, scale=2.2, limit=3.0)), (A | {"kv_from": 1}, moe(4, 1, 56, groups=(2, 1)))],
                     vocab=211, width=120, eps=3e-4, embed=1.7, mult=0.55),
    # nothing is a multiple of eight; two layers that read one layer's latents, seven taps
    "ragged": config([(B, moe(6, 2, 37, groups=(6, 3))), (forget(5, 13, 19), None), (B | {"kv_from": 0}, None), (forget(1, 7, 33), moe(3, 1, 29)),
                      (latent(3, 11, 5, rank=35, q_rank=50, rot=2, window=12), None), (B | {"kv_from": 0, "mask": {"size": 5}}, None)],
                     vocab=97, width=75, embed=0.9, taps=7, mult=1.3),
    # no routing: tight tolerances in 16 bits too
    "plain": config([(C, None), (forget(4, 16, 32), None), (C, None), (C | {"kv_from": 2}, None), (forget(2, 32, 32), None)], vocab=160, width=64, embed=3.0,
                    taps=3, mult=1.0),
    # heads as wide as the tensor-core prefill takes, whole state tiles and more
    "full": config([(D, None), (forget(2, 64, 64), None), (D | {"kv_from": 0, "mask": {"size": 33}}, None), (forget(1, 128, 96), None)], vocab=192, width=176),
    # wider than that; no window; a single tap; a row of more than 512 elements
    "wide": config([(E, None), (forget(1, 200, 48), None), (E | {"kv_from": 0, "mask": None}, None), (forget(1, 48, 232), None)], vocab=128, width=112, taps=1),
    # recurrent layers only, as many taps as there may be
    "state": config([(forget(2, 48, 48), moe(9, 4, 40, groups=(3, 2))), (forget(3, 20, 36), moe(1, 1, 24))], vocab=128, width=80, taps=16),
    # many heads of a token in a tile, a window of one token, two taps
    "alone": config([(latent(18, 16, 16, rank=24, q_rank=32, rot=4, window=1), None), (latent(20, 16, 16, rank=130, q_rank=16, rot=16, window=0), None)],
                    vocab=128, width=80, taps=2),
}
ROUTED = {"uneven", "ragged", "state"}


def make(name_or_config, seed=0):
    """(config, architecture, float32 weights holding bf16 values).  Norm weights, taps, bounds, gates and the coefficients of the
    average are spread out so that a swapped or missing one shows."""
    cfg = CASES[name_or_config] if isinstance(name_or_config, str) else name_or_config
    arch = FosulixArch.from_hf_config(cfg)
    w = random_weights(arch, seed=seed)
    g = torch.Generator().manual_seed(seed + 17)
    for k in w:
        shape, last = w[k].shape, k.rsplit(".", 1)[-1]
        if last in ("norm", "norm1", "norm2"):
            w[k] = 0.6 + 0.8 * torch.rand(shape, generator=g)
        elif last == "lower":
            w[k] = 0.95 * torch.rand(shape, generator=g)         # memories of one to many tokens
        elif last == "b":
            w[k] = 2.0 * torch.randn(shape, generator=g)
        elif last == "canon1":
            w[k] = 0.5 * torch.randn(shape, generator=g)
        elif last == "dwa":
            w[k] = 0.4 * torch.randn(shape, generator=g)
            w[k][-1] = 1.0
        elif k == "embed":
            w[k] = torch.randn(shape, generator=g) * arch.width ** -0.5 * 4.0
        elif last == "router":
            w[k] = w[k] * 1.5
        elif last in ("gate", "up"):
            w[k] = w[k] * 2.0                                    # gates and inputs past the bound
    return cfg, arch, {k: v.to(torch.bfloat16).float() for k, v in w.items()}
