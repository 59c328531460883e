"""Small Dolidra configurations and weights for the tests."""

import torch

from prism_infer_b200.models.architecture import DolidraArch
from prism_infer_b200.models.weights import random_weights
from replay_helpers import checkpoint, engine, error, portions, replay, tokens  # noqa: F401

SCALING = {"factor": 6.0, "low": 1.0, "high": 3.0, "original": 90}   # short wavelengths, ramp and long ones within a few pairs


def diff(heads, kv_heads, dim, vdim, window, *, rot, lam=0.5, base=3000.0, scaling=SCALING):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": 1.3 * dim ** -0.5, "diff": lam, "mask": {"size": window},
            "rot": {"base": base, "dims": rot, **({"scaling": scaling} if scaling else {})}}


def kept(heads, kv_heads, dim, vdim, window, keep, *, rot, base=800.0):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": 1.7 * dim ** -0.5,
            "mask": {"size": window, "keep_first": keep}, "rot": {"base": base, "dims": rot}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=0):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}, **({"shared": {"ff": shared}} if shared else {})}


def config(layers, *, vocab=200, width=96, side=24, loop=None, eps=1e-5):
    """``layers``: (mixer dictionary, feed-forward dictionary or None) per layer."""
    out = {"architecture": "Dolidra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "token_side": {"dim": side},
           "layers": [{"type": "attention" if "diff" in m else "attention_2", "mixer": m, "mlp": f} for m, f in layers]}
    if loop is not None:
        out["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return out


CASES = {
    # every size different, all kinds of feed-forward, a shared expert of one and a half times the routed width
    "uneven": config([(diff(3, 1, 24, 40, 19, rot=16, lam=0.35), dense(136)), (kept(4, 2, 40, 24, 11, 3, rot=24), moe(5, 2, 48, 72)),
                      (diff(6, 3, 16, 24, 33, rot=16, lam=0.8), None)], vocab=211, width=120, side=20, loop=(1, 3, 2), eps=3e-4),
    # nothing is a multiple of eight; more kept tokens than a key tile holds; key heads that are not shared
    "ragged": config([(kept(3, 3, 13, 7, 50, 70, rot=12), moe(7, 3, 37)), (diff(3, 3, 14, 19, 21, rot=6, scaling=None), dense(51))],
                     vocab=97, width=75, side=5, loop=(1, 2, 3)),
    # dense only, the loop covers every layer and runs once, groups of three heads, one kept token
    "once": config([(kept(6, 2, 32, 32, 17, 1, rot=32), dense(96)), (diff(6, 2, 32, 48, 30, rot=20), dense(64))], vocab=160, width=64,
                   loop=(0, 2, 1)),
    # the widest heads of the tensor-core prefill, no loop
    "full": config([(diff(4, 2, 128, 128, 70, rot=128), dense(160)), (kept(8, 1, 96, 128, 64, 5, rot=64), dense(80))], vocab=192, width=176),
    # heads wider than that, and wider than the tensor-core decode
    "wide": config([(diff(2, 1, 144, 176, 40, rot=144), None), (kept(2, 2, 272, 264, 25, 2, rot=100), dense(48))], vocab=128, width=112),
    # forty (head, map) rows over one key head; a window of one; one expert, top one
    "many": config([(diff(20, 1, 16, 16, 26, rot=8), moe(1, 1, 24, 24)), (kept(18, 1, 16, 32, 1, 0, rot=16), moe(9, 1, 40, 8))], vocab=128,
                   width=80, side=32, loop=(1, 2, 2)),
}
ROUTED = {"uneven", "ragged", "many"}


def make(name_or_config, seed=0):
    """(config, architecture, float32 weights holding bf16 values).  Norm weights and biases are spread out so that a
    swapped or missing one shows; the side table and the head are as large as the rest of the stream."""
    cfg = CASES[name_or_config] if isinstance(name_or_config, str) else name_or_config
    arch = DolidraArch.from_hf_config(cfg)
    w = random_weights(arch, seed=seed)
    g = torch.Generator().manual_seed(seed + 17)
    for k in w:
        if arch.init_kind(k) == "norm":
            w[k] = 0.6 + 0.8 * torch.rand(w[k].shape, generator=g)
        elif arch.init_kind(k) == "bias":
            w[k] = 0.4 * torch.randn(w[k].shape, generator=g)
        elif arch.init_kind(k) == "embedding":
            w[k] = torch.randn(w[k].shape, generator=g)
        elif k.endswith(".router"):
            w[k] = w[k] * 3.0
    w["head"] = w["head"] * 3.0
    return cfg, arch, {k: v.to(torch.bfloat16).float() for k, v in w.items()}
