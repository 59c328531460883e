"""Small Bokorax configurations and weights for the tests."""

import torch

from prism_infer_b200.models.architecture import BokoraxArch
from prism_infer_b200.models.weights import random_weights
from replay_helpers import checkpoint, engine, error, portions, replay, tokens  # noqa: F401


def tied(heads, kv_heads, dim, window, *, rot, base=900.0, slow=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": 1.6 * dim ** -0.5, "mask": {"size": window},
            "rot": {"base": base, "dims": rot, **({"scaling": {"factor": slow}} if slow else {})}}


def sink(heads, kv_heads, dim, vdim, *, rot, cap=4.0, base=4000.0, slow=None, kv_from=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": 1.4 * dim ** -0.5, "softcap": cap,
            "rot": {"base": base, "dims": rot, **({"scaling": {"factor": slow}} if slow else {})},
            **({"kv_from": kv_from} if kv_from is not None else {})}


def wkv(heads, dim):
    return {"heads": heads, "dim": dim}


def moe(experts, top, ff, *, identity=0, groups=None, scale=1.0, shared=0):
    return {"kind": "moe", "expert": {"ff": ff},
            "router": {"experts": experts, "top": top, "identity": identity, "scale": scale, "groups": {"count": (groups or (1, 1))[0],
                                                                                                       "keep": (groups or (1, 1))[1]}},
            **({"shared": {"ff": shared}} if shared else {})}


def kind(m):
    return "wkv" if "kv_heads" not in m else ("attention" if "mask" in m else "attention_2")


def config(layers, *, vocab=200, width=96, eps=1e-5, embed=2.0, logits=1.0):
    """``layers``: (mixer dictionary, feed-forward dictionary or None) per layer."""
    return {"architecture": "Bokorax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed},
            "logit_scale": logits, "layers": [{"type": kind(m), "mixer": m, "mlp": f} for m, f in layers]}


# name -> (configuration, rank of every recurrent layer's decay)
CASES = {
    # every size different, all mixers, keys of another layer, a shared expert of one and a half times the routed width
    "uneven": (config([(wkv(3, 24), moe(7, 3, 48, identity=2, groups=(3, 2), scale=1.7, shared=72)),
                       (sink(6, 2, 40, 24, rot=24, slow=3.0), moe(6, 2, 32, groups=(2, 1), scale=0.6, shared=32)),
                       (tied(4, 2, 32, 19, rot=20), None), (wkv(2, 40), None),
                       (sink(6, 2, 40, 24, rot=24, slow=3.0, cap=7.0, kv_from=1), moe(5, 2, 56, identity=3, scale=2.2))],
                      vocab=211, width=120, eps=3e-4, embed=1.7, logits=0.8), (12, 20)),
    # nothing is a multiple of eight; key heads that are not shared; two layers that read one layer's keys
    "ragged": (config([(sink(3, 3, 14, 7, rot=6), moe(4, 2, 37, identity=1, shared=21)), (wkv(5, 13), None),
                       (sink(3, 3, 14, 7, rot=6, kv_from=0), None), (tied(5, 1, 19, 33, rot=14, slow=2.5), moe(3, 1, 29)), (wkv(1, 7), None),
                       (sink(3, 3, 14, 7, rot=6, cap=1.5, kv_from=0), None)], vocab=97, width=75, embed=0.9, logits=3.0), (5, 11)),
    # no routing: tight tolerances in 16 bits too; one head of queries per head of keys, groups of three
    "plain": (config([(tied(6, 2, 32, 17, rot=32), None), (wkv(4, 16), None), (sink(4, 4, 24, 48, rot=8, cap=6.0), None), (wkv(2, 32), None)],
                     vocab=160, width=64, embed=3.0), (8, 24)),
    # the widest heads of the tensor-core prefill and whole state tiles
    "full": (config([(wkv(3, 64), None), (sink(8, 1, 128, 96, rot=64), None), (tied(4, 2, 128, 70, rot=128), None),
                     (sink(8, 1, 128, 96, rot=64, kv_from=1), None)], vocab=192, width=176), (32,)),
    # heads wider than that, and wider than the tensor-core decode
    "wide": (config([(wkv(2, 136), None), (sink(2, 1, 144, 176, rot=100, slow=6.0), None), (tied(2, 2, 264, 25, rot=264), None), (wkv(1, 200), None)],
                    vocab=128, width=112), (40, 3)),
    # recurrent layers only; a window of one token
    "state": (config([(wkv(2, 48), moe(9, 4, 40, identity=3, groups=(4, 3), shared=80)), (wkv(3, 20), moe(1, 1, 24))], vocab=128, width=80), (16, 9)),
    "alone": (config([(tied(18, 1, 16, 1, rot=16), None), (sink(20, 1, 16, 16, rot=16, cap=3.0), None)], vocab=128, width=80), ()),
}
ROUTED = {"uneven", "ragged", "state"}


def architecture(name_or_config, ranks=()):
    cfg, ranks = CASES[name_or_config] if isinstance(name_or_config, str) else (name_or_config, ranks)
    recurrent = [i for i, l in enumerate(cfg["layers"]) if l["type"] == "wkv"]
    arch = BokoraxArch.from_hf_config(cfg)
    return cfg, arch.with_tensor_shapes({f"l{i}.mix.w1": (r, cfg["width"]) for i, r in zip(recurrent, ranks)})


def make(name_or_config, ranks=(), seed=0):
    """(config, architecture, float32 weights holding bf16 values).  Norm weights, blends, decays, sinks and corrections are
    spread out so that a swapped or missing one shows."""
    cfg, arch = architecture(name_or_config, ranks)
    w = random_weights(arch, seed=seed)
    g = torch.Generator().manual_seed(seed + 17)
    for k in w:
        shape, last = w[k].shape, k.rsplit(".", 1)[-1]
        if last in ("norm1", "norm2") or k == "final.norm":
            w[k] = 0.8 * torch.rand(shape, generator=g) - 0.4
        elif last == "norm":
            w[k] = 0.6 + 0.8 * torch.rand(shape, generator=g)
        elif ".mu." in k:
            w[k] = torch.rand(shape, generator=g)
        elif last == "w0":
            w[k] = -4.0 + 4.5 * torch.rand(shape, generator=g)   # memories of one to a hundred tokens
        elif last in ("sink", "u"):
            w[k] = 1.5 * torch.randn(shape, generator=g)
        elif last == "correction":
            w[k] = 0.2 * torch.randn(shape, generator=g) - 0.3   # negative choice scores among them
        elif k == "embed":
            w[k] = torch.randn(shape, generator=g)
        elif last == "router":
            w[k] = w[k] * 1.5
        elif k.endswith("mix.w1") or k.endswith("mix.w2"):
            w[k] = w[k] * 2.0
    w["head"] = w["head"] * 3.0
    return cfg, arch, {k: v.to(torch.bfloat16).float() for k, v in w.items()}
