"""Model families (reference ``prism_infer/models/model_registry.py:10-35``): how ``config.json`` names
them, how it becomes an architecture description, which class runs it, which random-weight sizes exist and
which kernel units it needs.  An unknown name fails at start-up with the list of known ones rather than
somewhere inside weight loading."""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Callable, Mapping


@dataclass(frozen=True)
class ModelFamily:
    name: str
    multimodal: bool
    architecture_from_config: Callable[[Any], Any]
    model_class_path: str  # "module:Class", imported on demand
    random_architectures: Mapping[str, Callable[[], Any]] = field(default_factory=dict)  # names of "random:<name>" models
    float32_on_cuda: bool = False                  # the family has 32-bit kernels
    kv_modes: tuple[int, ...] = (0, 1, 2)          # cache element modes: dense, E4M3, scaled E4M3
    kernel_units: tuple[str, ...] = ()             # csrc/*.cu files it needs (empty: all of them)


def _qwen3_vl_arch(cfg: Any):
    from .architecture import Qwen3VLArch

    return Qwen3VLArch.from_hf_config(cfg)


def _qwen3_vl_random() -> dict[str, Callable[[], Any]]:
    from .architecture import Qwen3VLArch

    return {
        "tiny": Qwen3VLArch.tiny,
        "qwen3-vl-8b": Qwen3VLArch.qwen3_vl_8b,
        "qwen3_vl_8b": Qwen3VLArch.qwen3_vl_8b,
        "qwen3-vl-8b-2layer": Qwen3VLArch.qwen3_vl_8b_2layer,
        # profiling aids: the language-model compute of ONE rank of an n-way tensor-parallel group
        # (heads, KV heads, MLP width and vocabulary divided by n), run without any exchange
        "qwen3-vl-8b-tp2-shard": lambda: Qwen3VLArch.qwen3_vl_8b().rank_shard(2),
        "qwen3-vl-8b-tp4-shard": lambda: Qwen3VLArch.qwen3_vl_8b().rank_shard(4),
        "qwen3-vl-8b-tp8-shard": lambda: Qwen3VLArch.qwen3_vl_8b().rank_shard(8),
    }


def _poralorn_arch(cfg: Any):
    from .architecture import PoralornArch

    return PoralornArch.from_hf_config(cfg)


def _poralorn_random() -> dict[str, Callable[[], Any]]:
    from .architecture import PoralornArch

    return {"poralorn-tiny": PoralornArch.tiny, "poralorn-8b-like": lambda: PoralornArch.like_8b(36),
            "poralorn-8b-like-4layer": PoralornArch.like_8b}


def _dolidra_arch(cfg: Any):
    from .architecture import DolidraArch

    return DolidraArch.from_hf_config(cfg)


def _dolidra_random() -> dict[str, Callable[[], Any]]:
    from .architecture import DolidraArch

    return {"dolidra-tiny": DolidraArch.tiny, "dolidra-8b-like": lambda: DolidraArch.like_8b(36),
            "dolidra-8b-like-4layer": DolidraArch.like_8b}


def _bokorax_arch(cfg: Any):
    from .architecture import BokoraxArch

    return BokoraxArch.from_hf_config(cfg)


def _bokorax_random() -> dict[str, Callable[[], Any]]:
    from .architecture import BokoraxArch

    return {"bokorax-tiny": BokoraxArch.tiny, "bokorax-8b-like": lambda: BokoraxArch.like_8b(36),
            "bokorax-8b-like-4layer": BokoraxArch.like_8b}


def _fosulix_arch(cfg: Any):
    from .architecture import FosulixArch

    return FosulixArch.from_hf_config(cfg)


def _fosulix_random() -> dict[str, Callable[[], Any]]:
    from .architecture import FosulixArch

    return {"fosulix-tiny": FosulixArch.tiny, "fosulix-8b-like": lambda: FosulixArch.like_8b(36),
            "fosulix-8b-like-4layer": FosulixArch.like_8b}


_FAMILIES = {
    "qwen3_vl": ModelFamily("qwen3_vl", True, _qwen3_vl_arch, "prism_infer_b200.models.qwen3_vl:Qwen3VLModel", _qwen3_vl_random()),
    "poralorn": ModelFamily("poralorn", False, _poralorn_arch, "prism_infer_b200.models.poralorn:PoralornModel", _poralorn_random(),
                            float32_on_cuda=True, kv_modes=(0,),
                            kernel_units=("gemm_tcgen05", "gemm_f32", "attention_tcgen05", "latent_attention", "residual_stream",
                                          "kv_ops", "sampler")),
    "dolidra": ModelFamily("dolidra", False, _dolidra_arch, "prism_infer_b200.models.dolidra:DolidraModel", _dolidra_random(),
                           float32_on_cuda=True, kv_modes=(0,),
                           kernel_units=("gemm_tcgen05", "gemm_f32", "window_attention", "moe", "residual_stream", "kv_ops", "sampler")),
    "bokorax": ModelFamily("bokorax", False, _bokorax_arch, "prism_infer_b200.models.bokorax:BokoraxModel", _bokorax_random(),
                           float32_on_cuda=True, kv_modes=(0,),
                           kernel_units=("gemm_tcgen05", "gemm_f32", "window_attention", "recurrence", "moe", "residual_stream", "kv_ops",
                                         "sampler")),
    "fosulix": ModelFamily("fosulix", False, _fosulix_arch, "prism_infer_b200.models.fosulix:FosulixModel", _fosulix_random(),
                           float32_on_cuda=True, kv_modes=(0,),
                           kernel_units=("gemm_tcgen05", "gemm_f32", "latent_attention", "window_attention", "recurrence", "moe",
                                         "residual_stream", "kv_ops", "sampler")),
}


def known_model_types() -> list[str]:
    return sorted(_FAMILIES)


def resolve_model_family(model_type: str) -> ModelFamily:
    try:
        return _FAMILIES[model_type]
    except KeyError:
        raise ValueError(f"unsupported model_type {model_type!r}; supported: {known_model_types()}") from None


def family_of_config(cfg: Mapping[str, Any]) -> ModelFamily:
    """The family a ``config.json`` dictionary names: ``model_type``, or ``architecture`` in any spelling of case."""
    name = cfg.get("model_type")
    if name is None:
        name = str(cfg.get("architecture", "")).lower()
    return resolve_model_family(name)


def random_architecture(name: str):
    known = {n: make for fam in _FAMILIES.values() for n, make in fam.random_architectures.items()}
    if name not in known:
        raise ValueError(f"unknown random architecture {name!r}; known: {sorted(known)}")
    return known[name]()


def load_model_class(family: ModelFamily):
    import importlib

    module, _, cls = family.model_class_path.partition(":")
    return getattr(importlib.import_module(module), cls)
