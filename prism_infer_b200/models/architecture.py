"""Validated architecture descriptions, one frozen dataclass tree per model family.

The engine never reads a Hugging Face config object directly: it converts the
``config.json`` dictionary (or an ``AutoConfig`` instance) into the frozen
dataclasses below once and every later layer (weight sharding, kernels, KV sizing)
reads these.  Mirrors the contract of the reference's
``prism_infer/models/qwen3_vl_architecture.py:117-428`` (canonical 8B constants at
``:18-44``): interleaved M-RoPE only, no attention bias, SiLU text MLP, GELU-tanh
vision MLP.  ``PoralornArch``, ``DolidraArch``, ``BokoraxArch`` and ``FosulixArch`` (end of file) are text-only families: latent
attention, windowed attention with a mixture of experts, recurrent layers between attention layers, and gated linear attention
between windowed latent attention under a depth average.

What the engine asks of any architecture, whatever its family: ``model_type``, ``multimodal``,
``vocab_size``, ``max_positions`` (``None``: unbounded), ``num_layer_runs``, ``eos_token_id``, the
visual token ids (-1 where there are none), ``reserved_token_ids``, ``kv_geometry(tp)`` and ``state_sizes()``.
"""

from __future__ import annotations

import json
import math
import os
from dataclasses import asdict, dataclass, field, replace
from typing import Any, Mapping

SUPPORTED_MODEL_TYPES = frozenset({"qwen3_vl"})


@dataclass(frozen=True)
class KVGeometry:
    """Shape of one rank's paged cache: ``planes`` slabs per layer run (2: keys and values, 1: one row per token,
    a shared latent or all heads' keys and values), each ``[pages, heads, page, row]``.  ``rows`` gives every layer
    run a row width of its own (single plane, one head)."""

    planes: int
    layers: int
    heads: int
    row: int
    rows: tuple[int, ...] = ()

    def __post_init__(self) -> None:
        if self.rows and (self.planes != 1 or self.heads != 1 or len(self.rows) != self.layers or self.row != max(self.rows)):
            raise ValueError("row widths per layer run need a single-plane, single-head cache and one width per layer run")

    def bytes_per_page(self, page: int, element_bytes: int, scaled: bool = False) -> int:
        if self.rows:
            return sum(self.rows) * page * element_bytes
        rows = self.planes * self.layers * self.heads * page
        return rows * self.row * element_bytes + (rows * 4 if scaled else 0)


def _get(cfg: Any, *names: str, default: Any = ...) -> Any:
    for name in names:
        if isinstance(cfg, Mapping):
            if name in cfg:
                return cfg[name]
        elif hasattr(cfg, name):
            return getattr(cfg, name)
    if default is not ...:
        return default
    raise ValueError(f"Qwen3-VL config is missing required field {' or '.join(names)}")


@dataclass(frozen=True)
class TextArch:
    vocab_size: int = 151_936
    hidden_size: int = 4_096
    num_layers: int = 36
    num_heads: int = 32
    num_kv_heads: int = 8
    head_dim: int = 128
    intermediate_size: int = 12_288
    rope_theta: float = 5_000_000.0
    rms_norm_eps: float = 1.0e-6
    mrope_section: tuple[int, int, int] = (24, 20, 20)
    max_position_embeddings: int = 262_144
    tie_word_embeddings: bool = False

    def __post_init__(self) -> None:
        if self.num_heads % self.num_kv_heads:
            raise ValueError("num_heads must be a multiple of num_kv_heads")
        if self.head_dim % 2:
            raise ValueError("head_dim must be even")
        if sum(self.mrope_section) != self.head_dim // 2:
            raise ValueError(
                f"mrope_section {self.mrope_section} must sum to head_dim/2 = {self.head_dim // 2}"
            )
        if len(self.mrope_section) != 3:
            raise ValueError("mrope_section needs three entries (T, H, W)")

    @property
    def q_size(self) -> int:
        return self.num_heads * self.head_dim

    @property
    def kv_size(self) -> int:
        return self.num_kv_heads * self.head_dim


@dataclass(frozen=True)
class VisionArch:
    hidden_size: int = 1_152
    depth: int = 27
    num_heads: int = 16
    intermediate_size: int = 4_304
    in_channels: int = 3
    patch_size: int = 16
    temporal_patch_size: int = 2
    spatial_merge_size: int = 2
    num_position_embeddings: int = 2_304
    out_hidden_size: int = 4_096
    deepstack_visual_indexes: tuple[int, ...] = (8, 16, 24)
    rope_theta: float = 10_000.0
    layer_norm_eps: float = 1.0e-6

    def __post_init__(self) -> None:
        if self.hidden_size % self.num_heads:
            raise ValueError("vision hidden_size must be a multiple of num_heads")
        side = int(round(self.num_position_embeddings**0.5))
        if side * side != self.num_position_embeddings:
            raise ValueError("num_position_embeddings must be a perfect square")
        if (self.head_dim // 2) % 2:
            raise ValueError("vision head_dim/2 must be even for 2-D rotary embedding")
        for idx in self.deepstack_visual_indexes:
            if not 0 <= idx < self.depth:
                raise ValueError(f"deepstack index {idx} outside vision depth {self.depth}")

    @property
    def head_dim(self) -> int:
        return self.hidden_size // self.num_heads

    @property
    def patch_input_dim(self) -> int:
        return self.in_channels * self.temporal_patch_size * self.patch_size * self.patch_size

    @property
    def merge_unit(self) -> int:
        return self.spatial_merge_size * self.spatial_merge_size

    @property
    def merged_dim(self) -> int:
        return self.hidden_size * self.merge_unit

    @property
    def grid_per_side(self) -> int:
        return int(round(self.num_position_embeddings**0.5))


@dataclass(frozen=True)
class Qwen3VLArch:
    text: TextArch = field(default_factory=TextArch)
    vision: VisionArch = field(default_factory=VisionArch)
    image_token_id: int = 151_655
    video_token_id: int = 151_656
    vision_start_token_id: int = 151_652
    vision_end_token_id: int = 151_653
    eos_token_id: int = 151_645
    model_type: str = "qwen3_vl"

    def __post_init__(self) -> None:
        if self.model_type not in SUPPORTED_MODEL_TYPES:
            raise ValueError(f"unsupported model_type {self.model_type!r}")
        if self.vision.out_hidden_size != self.text.hidden_size:
            raise ValueError("vision out_hidden_size must equal text hidden_size")
        ids = (self.image_token_id, self.video_token_id, self.vision_start_token_id)
        if len(set(ids)) != 3:
            raise ValueError(f"visual special token ids must be distinct: {ids}")

    # ---- what the engine reads of every family ---------------------------------
    multimodal = True

    @property
    def vocab_size(self) -> int:
        return self.text.vocab_size

    @property
    def max_positions(self) -> int | None:
        return self.text.max_position_embeddings

    @property
    def num_layer_runs(self) -> int:
        return self.text.num_layers

    @property
    def reserved_token_ids(self) -> tuple[int, ...]:
        return (self.image_token_id, self.video_token_id, self.vision_start_token_id, self.vision_end_token_id, self.eos_token_id)

    def state_sizes(self) -> tuple[int, ...]:
        return ()

    def kv_geometry(self, tp: int = 1) -> KVGeometry:
        return KVGeometry(2, self.text.num_layers, self.text.num_kv_heads // tp, self.text.head_dim)

    # ---- factories -----------------------------------------------------------
    @classmethod
    def qwen3_vl_8b(cls) -> "Qwen3VLArch":
        return cls()

    def rank_shard(self, n: int) -> "Qwen3VLArch":
        """Architecture whose language model equals one rank's share of an ``n``-way
        tensor-parallel split (for single-GPU profiling of the per-rank kernel chain)."""
        import dataclasses

        validate_tensor_parallel(self, n)
        t = self.text
        text = dataclasses.replace(t, num_heads=t.num_heads // n, num_kv_heads=t.num_kv_heads // n,
                                   intermediate_size=t.intermediate_size // n, vocab_size=t.vocab_size // n)
        return dataclasses.replace(self, text=text)

    @classmethod
    def qwen3_vl_8b_2layer(cls) -> "Qwen3VLArch":
        """Qwen3-VL-8B widths (hidden 4096, 32 / 8 heads of 128, MLP 12288, vocabulary 151936, vision
        hidden 1152) with two decoder and two vision layers: every kernel runs at its production
        shape, and an end-to-end comparison against the oracle stays cheap."""
        import dataclasses

        full = cls()
        return dataclasses.replace(
            full, text=dataclasses.replace(full.text, num_layers=2),
            vision=dataclasses.replace(full.vision, depth=2, deepstack_visual_indexes=(0, 1)))

    @classmethod
    def tiny(cls) -> "Qwen3VLArch":
        """The small CPU test model: 2+2 layers, hidden 256/128, head_dim 64."""
        return cls(
            text=TextArch(
                vocab_size=1024,
                hidden_size=256,
                num_layers=2,
                num_heads=4,
                num_kv_heads=2,
                head_dim=64,
                intermediate_size=512,
                mrope_section=(8, 12, 12),
                max_position_embeddings=4096,
            ),
            vision=VisionArch(
                hidden_size=128,
                depth=2,
                num_heads=4,
                intermediate_size=256,
                num_position_embeddings=256,
                out_hidden_size=256,
                deepstack_visual_indexes=(1,),
            ),
            image_token_id=1001,
            video_token_id=1002,
            vision_start_token_id=1003,
            vision_end_token_id=1004,
            eos_token_id=1005,
        )

    @classmethod
    def from_hf_config(cls, cfg: Any) -> "Qwen3VLArch":
        model_type = _get(cfg, "model_type")
        if model_type not in SUPPORTED_MODEL_TYPES:
            raise ValueError(f"unsupported model_type {model_type!r}")
        tcfg = _get(cfg, "text_config")
        vcfg = _get(cfg, "vision_config")
        rope = _get(tcfg, "rope_scaling", "rope_parameters", default=None) or {}
        section = tuple(_get(rope, "mrope_section", default=(24, 20, 20)))
        if _get(rope, "mrope_interleaved", default=True) is False:
            raise ValueError("only interleaved M-RoPE is supported")
        if _get(tcfg, "attention_bias", default=False):
            raise ValueError("attention bias is not supported")
        if _get(tcfg, "hidden_act", default="silu") != "silu":
            raise ValueError("text MLP activation must be silu")
        vact = _get(vcfg, "hidden_act", default="gelu_pytorch_tanh")
        if vact not in ("gelu_pytorch_tanh", "gelu_tanh"):
            raise ValueError("vision MLP activation must be gelu (tanh)")
        theta = _get(tcfg, "rope_theta", default=None)
        if theta is None:
            theta = _get(rope, "rope_theta", default=5_000_000.0)
        hidden = int(_get(tcfg, "hidden_size"))
        heads = int(_get(tcfg, "num_attention_heads"))
        text = TextArch(
            vocab_size=int(_get(tcfg, "vocab_size")),
            hidden_size=hidden,
            num_layers=int(_get(tcfg, "num_hidden_layers")),
            num_heads=heads,
            num_kv_heads=int(_get(tcfg, "num_key_value_heads")),
            head_dim=int(_get(tcfg, "head_dim", default=hidden // heads)),
            intermediate_size=int(_get(tcfg, "intermediate_size")),
            rope_theta=float(theta),
            rms_norm_eps=float(_get(tcfg, "rms_norm_eps", default=1e-6)),
            mrope_section=section,  # type: ignore[arg-type]
            max_position_embeddings=int(_get(tcfg, "max_position_embeddings", default=262_144)),
            tie_word_embeddings=bool(
                _get(cfg, "tie_word_embeddings", default=_get(tcfg, "tie_word_embeddings", default=False))
            ),
        )
        vision = VisionArch(
            hidden_size=int(_get(vcfg, "hidden_size")),
            depth=int(_get(vcfg, "depth")),
            num_heads=int(_get(vcfg, "num_heads")),
            intermediate_size=int(_get(vcfg, "intermediate_size")),
            in_channels=int(_get(vcfg, "in_channels", default=3)),
            patch_size=int(_get(vcfg, "patch_size")),
            temporal_patch_size=int(_get(vcfg, "temporal_patch_size", default=2)),
            spatial_merge_size=int(_get(vcfg, "spatial_merge_size", default=2)),
            num_position_embeddings=int(_get(vcfg, "num_position_embeddings")),
            out_hidden_size=int(_get(vcfg, "out_hidden_size")),
            deepstack_visual_indexes=tuple(_get(vcfg, "deepstack_visual_indexes", default=(8, 16, 24))),
        )
        eos = _get(cfg, "eos_token_id", default=_get(tcfg, "eos_token_id", default=151_645))
        if isinstance(eos, (list, tuple)):
            eos = eos[0]
        return cls(
            text=text,
            vision=vision,
            image_token_id=int(_get(cfg, "image_token_id")),
            video_token_id=int(_get(cfg, "video_token_id")),
            vision_start_token_id=int(_get(cfg, "vision_start_token_id")),
            vision_end_token_id=int(_get(cfg, "vision_end_token_id", default=151_653)),
            eos_token_id=int(eos if eos is not None else 151_645),
            model_type=model_type,
        )

    @classmethod
    def from_pretrained(cls, path: str) -> "Qwen3VLArch":
        with open(os.path.join(path, "config.json"), "r", encoding="utf-8") as fh:
            return cls.from_hf_config(json.load(fh))

    def to_hf_config(self) -> dict[str, Any]:
        """A ``config.json`` dictionary Hugging Face ``AutoConfig`` accepts."""
        t, v = self.text, self.vision
        return {
            "architectures": ["Qwen3VLForConditionalGeneration"],
            "model_type": self.model_type,
            "image_token_id": self.image_token_id,
            "video_token_id": self.video_token_id,
            "vision_start_token_id": self.vision_start_token_id,
            "vision_end_token_id": self.vision_end_token_id,
            "tie_word_embeddings": t.tie_word_embeddings,
            "eos_token_id": self.eos_token_id,
            "text_config": {
                "model_type": "qwen3_vl_text",
                "vocab_size": t.vocab_size,
                "hidden_size": t.hidden_size,
                "num_hidden_layers": t.num_layers,
                "num_attention_heads": t.num_heads,
                "num_key_value_heads": t.num_kv_heads,
                "head_dim": t.head_dim,
                "intermediate_size": t.intermediate_size,
                "rope_theta": t.rope_theta,
                "rms_norm_eps": t.rms_norm_eps,
                "hidden_act": "silu",
                "attention_bias": False,
                "max_position_embeddings": t.max_position_embeddings,
                "rope_scaling": {
                    "mrope_interleaved": True,
                    "mrope_section": list(t.mrope_section),
                    "rope_type": "default",
                },
                "dtype": "bfloat16",
            },
            "vision_config": {
                "model_type": "qwen3_vl",
                "hidden_size": v.hidden_size,
                "depth": v.depth,
                "num_heads": v.num_heads,
                "intermediate_size": v.intermediate_size,
                "in_channels": v.in_channels,
                "patch_size": v.patch_size,
                "temporal_patch_size": v.temporal_patch_size,
                "spatial_merge_size": v.spatial_merge_size,
                "num_position_embeddings": v.num_position_embeddings,
                "out_hidden_size": v.out_hidden_size,
                "deepstack_visual_indexes": list(v.deepstack_visual_indexes),
                "hidden_act": "gelu_pytorch_tanh",
            },
        }

    def describe(self) -> dict[str, Any]:
        return asdict(self)


def validate_tensor_parallel(arch: Any, tp: int) -> None:
    """Every sharded dimension must divide evenly (reference ``engine/llm_engine.py:117-143``)."""
    if tp < 1:
        raise ValueError("tensor_parallel_size must be >= 1")
    if isinstance(arch, LoopedStack):
        if tp != 1:
            raise ValueError(f"the {type(arch).__name__.removesuffix('Arch')} family runs on one GPU (tensor_parallel_size 1)")
        return
    t = arch.text
    for name, value in (
        ("num_heads", t.num_heads),
        ("num_kv_heads", t.num_kv_heads),
        ("hidden_size", t.hidden_size),
        ("intermediate_size", t.intermediate_size),
        ("vocab_size", t.vocab_size),
    ):
        if value % tp:
            raise ValueError(f"tensor_parallel_size {tp} does not divide text {name}={value}")


# ----------------------------------------------------------------------- looped layer stacks
@dataclass(frozen=True)
class LayerRun:
    """One execution of a layer.  ``loop_pass`` is the pass number on the first layer of a pass of the looped
    section (where a loop input may be formed) and ``None`` elsewhere."""

    layer: int
    loop_pass: int | None = None


class LoopedStack:
    """What the text-only families with a looped section share: layers ``loop_start .. loop_stop - 1`` run
    ``loop_times`` times in a row (0: no looped section), every run with its own cache slab."""

    multimodal = False
    image_token_id = -1
    video_token_id = -1

    def check_stack(self) -> None:
        if self.vocab_size < 1 or self.width < 1 or not self.layers:
            raise ValueError("vocab, width and layers must be given")
        if self.loop_times < 0 or (self.has_loop and not 0 <= self.loop_start < self.loop_stop <= len(self.layers)):
            raise ValueError(f"loop {self.loop_start} .. {self.loop_stop} x {self.loop_times} does not fit {len(self.layers)} layers")
        if self.norm_eps < 0:
            raise ValueError("norm eps must not be negative")

    @property
    def has_loop(self) -> bool:
        return self.loop_times > 0

    @property
    def max_positions(self) -> int | None:
        return None                  # nothing bounds a position

    @property
    def reserved_token_ids(self) -> tuple[int, ...]:
        return ()

    def state_sizes(self) -> tuple[int, ...]:
        """fp32 elements that a sequence's recurrent state takes in each recurrent layer run (none: attention only)."""
        return ()

    def layer_runs(self) -> tuple[LayerRun, ...]:
        """Every layer execution in order; run ``i`` owns cache slab ``i``."""
        if not self.has_loop:
            return tuple(LayerRun(i) for i in range(len(self.layers)))
        runs = [LayerRun(i) for i in range(self.loop_start)]
        for t in range(self.loop_times):
            runs += [LayerRun(i, t if i == self.loop_start else None) for i in range(self.loop_start, self.loop_stop)]
        return tuple(runs + [LayerRun(i) for i in range(self.loop_stop, len(self.layers))])

    @property
    def num_layer_runs(self) -> int:
        return len(self.layer_runs())


def _field_reader(family: str):
    """``need(dictionary, key, where)``: a required field of a family's ``config.json``."""

    def need(d: Mapping[str, Any], key: str, where: str = "config") -> Any:
        if key not in d:
            raise ValueError(f"{family} {where} is missing required field {key}")
        return d[key]

    return need


def _loop_fields(cfg: Mapping[str, Any], need) -> dict[str, int]:
    loop = cfg.get("loop") or {}
    return {f"loop_{k}": int(need(loop, k, "loop")) if loop else 0 for k in ("start", "stop", "times")}


NO_WINDOW = 1 << 30              # a window that no sequence outgrows


# ------------------------------------------------------------------------------- Poralorn
@dataclass(frozen=True)
class LatentAttentionArch:
    """Sizes of one latent-attention mixer: ``heads`` heads whose ``dim``-wide keys and ``vdim``-wide values
    are linear in one shared ``kv_rank``-wide latent per token (the only thing cached).  ``q_rank``: the queries go through a
    normalised latent of their own (0: straight from the input); ``rot_dim`` more columns of every query, and of one key part
    all heads share (cached beside the latent), are rotated as ``rot`` says; a query sees the ``window`` newest positions;
    ``kv_from``: the layer whose cached rows it reads instead of its own (-1: none)."""

    heads: int
    dim: int
    vdim: int
    kv_rank: int
    scale: float
    q_rank: int = 0
    rot_dim: int = 0
    rot: RotaryArch | None = None
    window: int = NO_WINDOW
    kv_from: int = -1

    def __post_init__(self) -> None:
        for name in ("heads", "dim", "vdim", "kv_rank", "window"):
            if getattr(self, name) < 1:
                raise ValueError(f"latent attention: {name} must be positive")
        if self.q_rank < 0 or self.rot_dim < 0 or self.rot_dim != (self.rot.dims if self.rot is not None else 0):
            raise ValueError("latent attention: q_rank must not be negative, rot.dims is rot_dim")

    @property
    def rot_start(self) -> int:
        """Column of a query or key head at which its rotated part starts; ``dq`` the whole head, padded, ``dv`` a value head."""
        return -(-self.dim // 8) * 8

    @property
    def dq(self) -> int:
        return -(-(self.rot_start + self.rot_dim) // 16) * 16

    @property
    def dv(self) -> int:
        return -(-self.vdim // 16) * 16

    @property
    def row_rot_start(self) -> int:
        """Column of a cached row at which the rotated key part starts."""
        return -(-self.kv_rank // 16) * 16

    @property
    def cache_row(self) -> int:
        """Elements of a cached row, latent and rotated key part, in whole 64-element tiles."""
        return -(-(self.row_rot_start + self.rot_dim) // 64) * 64


@dataclass(frozen=True)
class PoralornLayer:
    mixer: LatentAttentionArch
    ff: int = 0                      # width of the feed-forward, 0: the layer has none


@dataclass(frozen=True)
class PoralornArch(LoopedStack):
    vocab_size: int
    width: int
    layers: tuple[PoralornLayer, ...]
    loop_start: int = 0              # layers loop_start .. loop_stop - 1 run loop_times times in a row
    loop_stop: int = 0
    loop_times: int = 0              # 0: no looped section
    norm_eps: float = 1.0e-5
    residual_mult: float = 1.0
    logit_softcap: float = 0.0       # 0: logits are not capped
    eos_token_id: int = -1
    model_type: str = "poralorn"

    def __post_init__(self) -> None:
        self.check_stack()
        if self.logit_softcap < 0:
            raise ValueError("logit_softcap must not be negative")

    # ---- what the engine reads of every family ---------------------------------
    @property
    def latent_row(self) -> int:
        """Elements of one cached latent row: the widest latent, rounded up to whole 64-element tiles."""
        return -(-max(l.mixer.kv_rank for l in self.layers) // 64) * 64

    def kv_geometry(self, tp: int = 1) -> KVGeometry:
        return KVGeometry(1, self.num_layer_runs, 1, self.latent_row)

    # ---- checkpoint --------------------------------------------------------------
    def weight_shapes(self) -> dict[str, tuple[int, ...]]:
        s: dict[str, tuple[int, ...]] = {"embed": (self.vocab_size, self.width)}
        if self.has_loop:
            s["loop.in"] = (self.width, 2 * self.width)
            s["loop.step"] = (self.loop_times, self.width)
        for i, l in enumerate(self.layers):
            m, p = l.mixer, f"l{i}"
            s[f"{p}.norm1"] = ()
            s[f"{p}.mix.q"] = (m.heads * m.dim, self.width)
            s[f"{p}.mix.dkv"] = (m.kv_rank, self.width)
            s[f"{p}.mix.dkv.norm"] = (m.kv_rank,)
            s[f"{p}.mix.uk"] = (m.heads * m.dim, m.kv_rank)
            s[f"{p}.mix.uv"] = (m.heads * m.vdim, m.kv_rank)
            s[f"{p}.mix.g"] = (m.heads * m.vdim, self.width)
            s[f"{p}.mix.o"] = (self.width, m.heads * m.vdim)
            s[f"{p}.rg1"] = (self.width, self.width)
            s[f"{p}.rg1.b"] = (self.width,)
            if l.ff:
                s[f"{p}.norm2"] = ()
                s[f"{p}.mlp.up"] = (l.ff, self.width)
                s[f"{p}.mlp.down"] = (self.width, l.ff)
                s[f"{p}.rg2"] = (self.width, self.width)
                s[f"{p}.rg2.b"] = (self.width,)
        s["final.norm"] = ()
        s["head"] = (self.vocab_size, self.width)
        return s

    @staticmethod
    def init_kind(name: str) -> str:
        """How random initialisation draws a tensor: ``norm``, ``bias``, ``embedding`` or ``matrix``."""
        if name.rsplit(".", 1)[-1] in ("norm", "norm1", "norm2"):
            return "norm"
        if name.endswith(".b") or name == "loop.step":
            return "bias"
        return "embedding" if name == "embed" else "matrix"

    # ---- factories ---------------------------------------------------------------
    @classmethod
    def from_hf_config(cls, cfg: Mapping[str, Any]) -> "PoralornArch":
        """From the ``config.json`` dictionary."""
        need = _field_reader("Poralorn")
        layers = []
        for i, entry in enumerate(need(cfg, "layers")):
            where = f"layer {i}"
            kind = need(entry, "type", where)
            if kind != "latent_attention":
                raise ValueError(f"Poralorn {where}: unsupported mixer {kind!r}")
            m = need(entry, "mixer", where)
            mixer = LatentAttentionArch(*(int(need(m, k, where)) for k in ("heads", "dim", "vdim", "kv_rank")),
                                        float(need(m, "scale", where)))
            mlp = entry.get("mlp")
            if mlp is not None and mlp.get("kind") != "dense":
                raise ValueError(f"Poralorn {where}: unsupported feed-forward {mlp.get('kind')!r}")
            layers.append(PoralornLayer(mixer, int(need(mlp, "ff", where)) if mlp is not None else 0))
        return cls(
            vocab_size=int(need(cfg, "vocab")), width=int(need(cfg, "width")), layers=tuple(layers), **_loop_fields(cfg, need),
            norm_eps=float(need(need(cfg, "norm"), "eps", "norm")), residual_mult=float(need(cfg, "residual_mult")),
            logit_softcap=float(cfg.get("logit_softcap") or 0.0))

    def to_hf_config(self) -> dict[str, Any]:
        """The ``config.json`` dictionary ``from_hf_config`` reads."""
        out: dict[str, Any] = {"architecture": "Poralorn", "vocab": self.vocab_size, "width": self.width,
                               "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult,
                               "logit_softcap": self.logit_softcap,
                               "layers": [{"type": "latent_attention",
                                           "mixer": {k: getattr(l.mixer, k) for k in ("heads", "dim", "vdim", "kv_rank", "scale")},
                                           "mlp": {"kind": "dense", "ff": l.ff} if l.ff else None} for l in self.layers]}
        if self.has_loop:
            out["loop"] = {"start": self.loop_start, "stop": self.loop_stop, "times": self.loop_times}
        return out

    @classmethod
    def tiny(cls) -> "PoralornArch":
        """The small CPU test model: five layer runs, every size different."""
        mixers = (LatentAttentionArch(3, 32, 24, 40, 0.17), LatentAttentionArch(5, 16, 16, 72, 0.25))
        return cls(vocab_size=300, width=160, layers=(PoralornLayer(mixers[0], 208), PoralornLayer(mixers[1]), PoralornLayer(mixers[0], 96)),
                   loop_start=1, loop_stop=2, loop_times=3, norm_eps=1e-5, residual_mult=0.4, logit_softcap=12.0)

    @classmethod
    def like_8b(cls, layers: int = 4, *, width: int = 4096, heads: int = 32, dim: int = 128, kv_rank: int = 512,
                ff: int = 12288, vocab_size: int = 151_936) -> "PoralornArch":
        """Layers with the widths of an 8B-class decoder (measurement model; random weights)."""
        mixer = LatentAttentionArch(heads, dim, dim, kv_rank, dim ** -0.5)
        return cls(vocab_size=vocab_size, width=width, layers=(PoralornLayer(mixer, ff),) * layers, residual_mult=0.5,
                   logit_softcap=30.0)


# -------------------------------------------------------------------------------- Dolidra
@dataclass(frozen=True)
class RotaryArch:
    """Rotation of the first ``dims`` columns of a head (pairs ``(i, i + dims / 2)``, or neighbours where the mixer says so).
    ``factor`` > 0 rescales the frequencies by wavelength: long ones are divided by it, those below ``original / high`` stay, a
    ramp between; without ``original`` all of them are divided.  With ``fast`` and ``slow`` (turns over ``original`` positions)
    the ramp is over the pairs' numbers instead (YaRN), and sines and cosines are scaled by ``amplitude``."""

    base: float
    dims: int
    factor: float = 0.0
    low: float = 0.0
    high: float = 0.0
    original: float = 0.0
    fast: float = 0.0
    slow: float = 0.0

    def __post_init__(self) -> None:
        if self.dims < 0 or self.dims % 2:
            raise ValueError(f"rotary dims must be even, got {self.dims}")
        if self.fast > 0.0 and not (self.slow > 0.0 and self.factor > 0.0 and self.original > 0.0 and self.base > 1.0):
            raise ValueError("rotary scaling by turns needs factor, original, fast and slow, and a base above one")

    @property
    def amplitude(self) -> float:
        return 0.1 * math.log(self.factor) + 1.0 if self.fast > 0.0 else 1.0

    def _by_turns(self) -> list[float]:
        """The frequencies with those of slow pairs divided by ``factor``, a ramp over the pairs' numbers between."""

        def pair(turns: float) -> float:
            return self.dims * math.log(self.original / (2.0 * math.pi * turns)) / (2.0 * math.log(self.base))

        lo, hi = max(math.floor(pair(self.fast)), 0), min(math.ceil(pair(self.slow)), self.dims - 1)
        out = []
        for i in range(self.dims // 2):
            f, ramp = self.base ** (-2.0 * i / self.dims), min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            out.append(f / self.factor * ramp + f * (1.0 - ramp))
        return out

    def inv_freq(self) -> list[float]:
        if self.fast > 0.0:
            return self._by_turns()
        out = []
        for i in range(self.dims // 2):
            f = self.base ** (-2.0 * i / self.dims)
            if self.factor > 0.0 and self.original == 0.0:
                f /= self.factor
            elif self.factor > 0.0:
                wavelength = 2.0 * math.pi / f
                if wavelength > self.original / self.low:
                    f /= self.factor
                elif wavelength >= self.original / self.high:
                    keep = (self.original / wavelength - self.low) / (self.high - self.low)
                    f = (1.0 - keep) * f / self.factor + keep * f
            out.append(f)
        return out


@dataclass(frozen=True)
class WindowAttentionArch:
    """One windowed attention mixer.  ``maps`` 2: differential attention (two maps over the same values, the second
    subtracted); ``qk_norm``: RMS norm over the whole query and the whole key projection, or (``head_norm``) over every
    head with one weight for all; ``gate``: one sigmoid output gate per head; a query sees the ``window`` newest positions
    (its own included) and the first ``keep_first``.  ``tied_values``: the values are the keys as projected; ``softcap``
    bounds the scores (0: no bound); ``sink``: a learned score per head in the softmax's denominator; ``kv_from``: the layer
    whose cached keys and values it reads instead of its own (-1: none)."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: RotaryArch
    window: int
    keep_first: int = 0
    maps: int = 1
    diff: float = 0.0
    bias: bool = False
    qk_norm: bool = False
    gate: bool = False
    head_norm: bool = False
    tied_values: bool = False
    softcap: float = 0.0
    sink: bool = False
    kv_from: int = -1

    def __post_init__(self) -> None:
        for name in ("heads", "kv_heads", "dim", "vdim", "window"):
            if getattr(self, name) < 1:
                raise ValueError(f"windowed attention: {name} must be positive")
        if self.heads % self.kv_heads:
            raise ValueError(f"windowed attention: {self.heads} query heads over {self.kv_heads} key/value heads")
        if self.rot.dims > self.dim or self.keep_first < 0 or self.maps not in (1, 2):
            raise ValueError("windowed attention: rot.dims must not exceed dim, keep_first must not be negative, maps is 1 or 2")
        if self.tied_values and (self.vdim != self.dim or self.maps != 1):
            raise ValueError("windowed attention: values that are the keys have the keys' width, and one map")
        if self.softcap < 0.0:
            raise ValueError("windowed attention: softcap must not be negative")

    @property
    def dq(self) -> int:
        """Key width of one map of one head, padded to whole tensor-core steps; ``dv`` likewise for values."""
        return -(-self.dim // 16) * 16

    @property
    def dv(self) -> int:
        return -(-self.vdim // 16) * 16

    @property
    def cache_row(self) -> int:
        """Elements a token's keys and values take: ``[key heads x maps x dq | value heads x dv]``."""
        return self.kv_heads * (self.maps * self.dq + self.dv)


@dataclass(frozen=True)
class MixtureArch:
    """Routed experts: ``top`` of ``experts`` gated feed-forwards of width ``ff`` per token, and one of width
    ``shared_ff`` (0: none) for every token, times a sigmoid per token with ``shared_gate``.  The weights are the softmax over
    the chosen logits, or (``scored``) the chosen scores of a softmax over all, divided by their sum and times ``scale``; then
    a learned correction enters the choice only, ``identity`` more router outputs stand for the input itself, and the
    choice is among the ``groups_kept`` best of ``groups`` equal groups of neighbours.  ``sigmoid``: the scores are the outputs'
    own sigmoids instead, not corrected and not divided by their sum, and a group is as good as the sum of its two best.
    ``limit``: the experts' gates and inputs are bounded (``act(min(g, limit)) * (1 + clamp(u, -limit, limit))``); 0: SiLU."""

    experts: int
    top: int
    ff: int
    shared_ff: int = 0
    scored: bool = False
    identity: int = 0
    groups: int = 1
    groups_kept: int = 1
    scale: float = 1.0
    shared_gate: bool = False
    sigmoid: bool = False
    limit: float = 0.0

    @property
    def outputs(self) -> int:
        """Router outputs that can be chosen."""
        return self.experts + self.identity

    def __post_init__(self) -> None:
        if self.experts < 1 or not 1 <= self.top <= self.outputs or self.ff < 1 or self.shared_ff < 0 or self.identity < 0:
            raise ValueError(f"mixture of experts: {self.top} of {self.experts} experts of width {self.ff}, shared {self.shared_ff}")
        if not 1 <= self.groups_kept <= self.groups or self.outputs % self.groups or self.top > self.outputs // self.groups * self.groups_kept:
            raise ValueError(f"mixture of experts: {self.top} of {self.outputs} in {self.groups_kept} of {self.groups} groups")
        if not self.scored and (self.identity or self.groups > 1 or self.scale != 1.0):
            raise ValueError("mixture of experts: identity experts, groups and a scale belong to scored routing")
        if (self.sigmoid and not self.scored) or self.limit < 0.0:
            raise ValueError("mixture of experts: sigmoid scores belong to scored routing, a limit must not be negative")


@dataclass(frozen=True)
class DolidraLayer:
    mixer: WindowAttentionArch
    ff: int = 0                      # width of a dense feed-forward
    moe: MixtureArch | None = None   # or a mixture; neither: the layer has no feed-forward

    @property
    def has_ff(self) -> bool:
        return self.ff > 0 or self.moe is not None


@dataclass(frozen=True)
class DolidraArch(LoopedStack):
    vocab_size: int
    width: int
    layers: tuple[DolidraLayer, ...]
    side_dim: int                    # width of a layer's part of the per-token side table
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 0
    norm_eps: float = 1.0e-5
    eos_token_id: int = -1
    model_type: str = "dolidra"

    def __post_init__(self) -> None:
        self.check_stack()
        if self.side_dim < 1:
            raise ValueError("token_side.dim must be positive")

    def kv_geometry(self, tp: int = 1) -> KVGeometry:
        rows = tuple(self.layers[r.layer].mixer.cache_row for r in self.layer_runs())
        return KVGeometry(1, len(rows), 1, max(rows), rows)

    # ---- checkpoint --------------------------------------------------------------
    def weight_shapes(self) -> dict[str, tuple[int, ...]]:
        W, D = self.width, self.side_dim
        s: dict[str, tuple[int, ...]] = {"embed": (self.vocab_size, W), "side.embed": (self.vocab_size, len(self.layers) * D)}

        def ff(prefix: str, width: int) -> None:
            s[f"{prefix}.gate"] = s[f"{prefix}.up"] = (width, W)
            s[f"{prefix}.down"] = (W, width)

        for i, l in enumerate(self.layers):
            m, p = l.mixer, f"l{i}"
            for n in ("norm1", "norm1b") + (("norm2", "norm2b") if l.has_ff else ()):
                s[f"{p}.{n}"] = (W,)
            sizes = {"q": m.heads * m.maps * m.dim, "k": m.kv_heads * m.maps * m.dim, "v": m.kv_heads * m.vdim}
            for n, rows in sizes.items():
                s[f"{p}.mix.{n}"] = (rows, W)
                if m.bias:
                    s[f"{p}.mix.{n}.b"] = (rows,)
            if m.maps == 2:
                for n in ("lq1", "lk1", "lq2", "lk2"):
                    s[f"{p}.mix.{n}"] = (m.dim,)
            if m.qk_norm:
                s[f"{p}.mix.q.norm"], s[f"{p}.mix.k.norm"] = (sizes["q"],), (sizes["k"],)
            if m.gate:
                s[f"{p}.mix.g"] = (m.heads, W)
            s[f"{p}.mix.o"] = (W, m.heads * m.vdim)
            if l.moe is not None:
                s[f"{p}.mlp.router"] = (l.moe.experts, W)
                for e in range(l.moe.experts):
                    ff(f"{p}.mlp.e{e}", l.moe.ff)
                if l.moe.shared_ff:
                    ff(f"{p}.mlp.shared", l.moe.shared_ff)
            elif l.ff:
                ff(f"{p}.mlp", l.ff)
            s[f"{p}.side.gate"], s[f"{p}.side.proj"], s[f"{p}.side.norm"] = (D, W), (W, D), (W,)
        s["final.norm"] = (W,)
        s["head"] = (self.vocab_size, W)
        return s

    @staticmethod
    def init_kind(name: str) -> str:
        """How random initialisation draws a tensor: ``norm``, ``bias``, ``embedding`` or ``matrix``."""
        last = name.rsplit(".", 1)[-1]
        if last.startswith("norm"):
            return "norm"
        if last in ("b", "lq1", "lk1", "lq2", "lk2"):
            return "bias"
        return "embedding" if name in ("embed", "side.embed") else "matrix"

    # ---- factories ---------------------------------------------------------------
    @classmethod
    def from_hf_config(cls, cfg: Mapping[str, Any]) -> "DolidraArch":
        """From the ``config.json`` dictionary."""
        need = _field_reader("Dolidra")
        layers = []
        for i, entry in enumerate(need(cfg, "layers")):
            where = f"layer {i}"
            kind = need(entry, "type", where)
            if kind not in ("attention", "attention_2"):
                raise ValueError(f"Dolidra {where}: unsupported mixer {kind!r}")
            m = need(entry, "mixer", where)
            rot, mask = need(m, "rot", where), need(m, "mask", where)
            scaling = rot.get("scaling") or {}
            rotary = RotaryArch(float(need(rot, "base", where)), int(need(rot, "dims", where)),
                                *(float(need(scaling, k, where)) for k in ("factor", "low", "high", "original")) if scaling else ())
            common = dict(heads=int(need(m, "heads", where)), kv_heads=int(need(m, "kv_heads", where)), dim=int(need(m, "dim", where)),
                          vdim=int(need(m, "vdim", where)), scale=float(need(m, "scale", where)), rot=rotary,
                          window=int(need(mask, "size", where)), keep_first=int(mask.get("keep_first") or 0))
            if kind == "attention":
                mixer = WindowAttentionArch(**common, maps=2, diff=float(need(m, "diff", where)), bias=True)
            else:
                mixer = WindowAttentionArch(**common, qk_norm=True, gate=True)
            mlp = entry.get("mlp")
            if mlp is None:
                layers.append(DolidraLayer(mixer))
            elif mlp.get("kind") == "dense":
                layers.append(DolidraLayer(mixer, ff=int(need(mlp, "ff", where))))
            elif mlp.get("kind") == "moe":
                router, shared = need(mlp, "router", where), mlp.get("shared") or {}
                layers.append(DolidraLayer(mixer, moe=MixtureArch(
                    int(need(router, "experts", where)), int(need(router, "top", where)), int(need(need(mlp, "expert", where), "ff", where)),
                    int(need(shared, "ff", where)) if shared else 0)))
            else:
                raise ValueError(f"Dolidra {where}: unsupported feed-forward {mlp.get('kind')!r}")
        return cls(vocab_size=int(need(cfg, "vocab")), width=int(need(cfg, "width")), layers=tuple(layers),
                   side_dim=int(need(need(cfg, "token_side"), "dim", "token_side")), **_loop_fields(cfg, need),
                   norm_eps=float(need(need(cfg, "norm"), "eps", "norm")))

    def to_hf_config(self) -> dict[str, Any]:
        """The ``config.json`` dictionary ``from_hf_config`` reads."""

        def layer(l: DolidraLayer) -> dict[str, Any]:
            m, r = l.mixer, l.mixer.rot
            rot: dict[str, Any] = {"base": r.base, "dims": r.dims}
            if r.factor > 0.0:
                rot["scaling"] = {"factor": r.factor, "low": r.low, "high": r.high, "original": r.original}
            mixer: dict[str, Any] = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "rot": rot,
                                     "mask": {"size": m.window}}
            if m.maps == 2:
                mixer["diff"] = m.diff
            if m.keep_first or m.maps == 1:
                mixer["mask"]["keep_first"] = m.keep_first
            mlp: dict[str, Any] | None = {"kind": "dense", "ff": l.ff} if l.ff else None
            if l.moe is not None:
                mlp = {"kind": "moe", "router": {"experts": l.moe.experts, "top": l.moe.top}, "expert": {"ff": l.moe.ff}}
                if l.moe.shared_ff:
                    mlp["shared"] = {"ff": l.moe.shared_ff}
            return {"type": "attention" if m.maps == 2 else "attention_2", "mixer": mixer, "mlp": mlp}

        out: dict[str, Any] = {"architecture": "Dolidra", "vocab": self.vocab_size, "width": self.width, "norm": {"eps": self.norm_eps},
                               "token_side": {"dim": self.side_dim}, "layers": [layer(l) for l in self.layers]}
        if self.has_loop:
            out["loop"] = {"start": self.loop_start, "stop": self.loop_stop, "times": self.loop_times}
        return out

    @classmethod
    def tiny(cls) -> "DolidraArch":
        """The small CPU test model: every size different, both mixers, all three kinds of feed-forward, five layer runs."""
        scaled = RotaryArch(20000.0, 24, 4.0, 1.0, 4.0, 64.0)
        diff = WindowAttentionArch(3, 1, 24, 40, 0.2, scaled, window=19, maps=2, diff=0.45, bias=True)
        kept = WindowAttentionArch(4, 2, 32, 16, 0.17, RotaryArch(5000.0, 8), window=11, keep_first=3, qk_norm=True, gate=True)
        return cls(vocab_size=310, width=144, side_dim=20, layers=(DolidraLayer(diff, ff=176), DolidraLayer(kept, moe=MixtureArch(5, 2, 48, 72)),
                                                                   DolidraLayer(diff)), loop_start=1, loop_stop=2, loop_times=3)

    @classmethod
    def like_8b(cls, layers: int = 4, *, width: int = 4096, heads: int = 16, kv_heads: int = 4, dim: int = 128, window: int = 1024,
                ff: int = 12288, experts: int = 32, top: int = 4, expert_ff: int = 1536, side_dim: int = 256,
                vocab_size: int = 151_936) -> "DolidraArch":
        """Layers with the widths of an 8B-class decoder (measurement model; random weights): differential layers with
        dense and with routed feed-forwards in turn, every fourth layer with kept first tokens and twice the heads."""
        rot = RotaryArch(1.0e6, dim, 8.0, 1.0, 4.0, 8192.0)
        diff = WindowAttentionArch(heads, kv_heads, dim, dim, dim ** -0.5, rot, window=window, maps=2, diff=0.6, bias=True)
        kept = WindowAttentionArch(2 * heads, 2 * kv_heads, dim, dim, dim ** -0.5, RotaryArch(1.0e6, dim), window=window, keep_first=16,
                                   qk_norm=True, gate=True)
        moe = MixtureArch(experts, top, expert_ff, expert_ff)
        kinds = [DolidraLayer(kept if i % 4 == 2 else diff, **({"moe": moe} if i % 2 else {"ff": ff})) for i in range(layers)]
        return cls(vocab_size=vocab_size, width=width, layers=tuple(kinds), side_dim=side_dim)


# -------------------------------------------------------------------------------- Bokorax
@dataclass(frozen=True)
class TimeMixArch:
    """A recurrent mixer with a matrix state per head (``dim`` x ``dim``): decay per key channel, data-dependent through a
    projection of rank ``decay_rank`` (a checkpoint's tensor shapes give it), and a bonus for the current token.  Every
    projection reads its own blend of the token's row and the previous token's."""

    heads: int
    dim: int
    decay_rank: int = 64

    def __post_init__(self) -> None:
        if self.heads < 1 or self.dim < 1 or self.decay_rank < 1:
            raise ValueError(f"time mixing: {self.heads} heads of {self.dim}, decay rank {self.decay_rank}")

    @property
    def dp(self) -> int:
        """Head width padded to whole tensor-core steps."""
        return -(-self.dim // 16) * 16

    def state_size(self, width: int) -> int:
        """fp32 elements of a sequence's state: ``[heads, dp, dp]`` and the previous token's row."""
        return self.heads * self.dp * self.dp + -(-width // 16) * 16


@dataclass(frozen=True)
class BokoraxLayer:
    mixer: WindowAttentionArch | TimeMixArch
    moe: MixtureArch | None = None

    @property
    def recurrent(self) -> bool:
        return isinstance(self.mixer, TimeMixArch)

    @property
    def owns_cache(self) -> bool:
        return not self.recurrent and self.mixer.kv_from < 0


@dataclass(frozen=True)
class BokoraxArch(LoopedStack):
    vocab_size: int
    width: int
    layers: tuple[BokoraxLayer, ...]
    embed_scale: float = 1.0
    logit_scale: float = 1.0
    norm_eps: float = 1.0e-6
    eos_token_id: int = -1
    model_type: str = "bokorax"

    loop_start = loop_stop = loop_times = 0   # every layer runs once

    def __post_init__(self) -> None:
        self.check_stack()
        for i, l in enumerate(self.layers):
            if l.recurrent or l.owns_cache:
                continue
            m, j = l.mixer, l.mixer.kv_from
            owner = self.layers[j] if j < i else None
            if owner is None or not owner.owns_cache:
                raise ValueError(f"Bokorax layer {i}: kv_from {j} does not name an earlier layer with keys of its own")
            if (m.kv_heads, m.dim, m.vdim) != (owner.mixer.kv_heads, owner.mixer.dim, owner.mixer.vdim):
                raise ValueError(f"Bokorax layer {i}: keys and values of layer {j} have other sizes")

    def cache_slab(self, layer: int) -> int:
        """Cache slab a layer's attention reads (-1: a recurrent layer)."""
        l = self.layers[layer]
        if l.recurrent:
            return -1
        owner = layer if l.owns_cache else l.mixer.kv_from
        return sum(o.owns_cache for o in self.layers[:owner])

    def state_slab(self, layer: int) -> int:
        return sum(l.recurrent for l in self.layers[:layer]) if self.layers[layer].recurrent else -1

    def kv_geometry(self, tp: int = 1) -> KVGeometry:
        rows = tuple(l.mixer.cache_row for l in self.layers if l.owns_cache) or (16,)   # pages count tokens even without keys
        return KVGeometry(1, len(rows), 1, max(rows), rows)

    def state_sizes(self) -> tuple[int, ...]:
        return tuple(l.mixer.state_size(self.width) for l in self.layers if l.recurrent)

    # ---- checkpoint --------------------------------------------------------------
    def weight_shapes(self) -> dict[str, tuple[int, ...]]:
        W = self.width
        s: dict[str, tuple[int, ...]] = {"embed": (self.vocab_size, W)}

        def ff(prefix: str, width: int) -> None:
            s[f"{prefix}.gate"] = s[f"{prefix}.up"] = (width, W)
            s[f"{prefix}.down"] = (W, width)

        for i, l in enumerate(self.layers):
            m, p = l.mixer, f"l{i}"
            s[f"{p}.norm1"] = (W,)
            if l.recurrent:
                C = m.heads * m.dim
                for n in "rkvgw":
                    s[f"{p}.mix.mu.{n}"] = (W,)
                for n in "rkvg":
                    s[f"{p}.mix.{n}"] = (C, W)
                s[f"{p}.mix.w1"], s[f"{p}.mix.w2"], s[f"{p}.mix.w0"] = (m.decay_rank, W), (C, m.decay_rank), (C,)
                s[f"{p}.mix.u"], s[f"{p}.mix.norm"], s[f"{p}.mix.o"] = (m.heads, m.dim), (C,), (W, C)
            else:
                sizes = {"q": m.heads * m.dim}
                if m.kv_from < 0:
                    sizes["k"] = m.kv_heads * m.dim
                    if not m.tied_values:
                        sizes["v"] = m.kv_heads * m.vdim
                for n, rows in sizes.items():
                    s[f"{p}.mix.{n}"] = (rows, W)
                    if m.qk_norm and n != "v":
                        s[f"{p}.mix.{n}.norm"] = (m.dim if m.head_norm else rows,)
                if m.sink:
                    s[f"{p}.mix.sink"] = (m.heads,)
                if m.gate:
                    s[f"{p}.mix.g"] = (m.heads, W)
                s[f"{p}.mix.o"] = (W, m.heads * m.vdim)
            if l.moe is not None:
                s[f"{p}.norm2"] = (W,)
                s[f"{p}.mlp.router"], s[f"{p}.mlp.correction"] = (l.moe.outputs, W), (l.moe.outputs,)
                for e in range(l.moe.experts):
                    ff(f"{p}.mlp.e{e}", l.moe.ff)
                if l.moe.shared_ff:
                    ff(f"{p}.mlp.shared", l.moe.shared_ff)
                    s[f"{p}.mlp.shared.sg"] = (1, W)
        s["final.norm"] = (W,)
        s["head"] = (self.vocab_size, W)
        return s

    def with_tensor_shapes(self, shapes: Mapping[str, tuple[int, ...]]) -> "BokoraxArch":
        """The sizes that only a checkpoint's tensors tell: the rank of every decay projection."""
        def sized(i: int, l: BokoraxLayer) -> BokoraxLayer:
            shape = shapes.get(f"l{i}.mix.w1") if l.recurrent else None
            return replace(l, mixer=replace(l.mixer, decay_rank=int(shape[0]))) if shape else l

        return replace(self, layers=tuple(sized(i, l) for i, l in enumerate(self.layers)))

    @staticmethod
    def init_kind(name: str) -> str:
        """How random initialisation draws a tensor: ``norm``, ``bias``, ``embedding`` or ``matrix``."""
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1", "norm2", "w0", "u", "sink", "correction") or name == "final.norm" or ".mu." in name:
            return "bias"            # norm weights around zero among them
        if last == "norm":
            return "norm"
        return "embedding" if name == "embed" else "matrix"

    # ---- factories ---------------------------------------------------------------
    @classmethod
    def from_hf_config(cls, cfg: Mapping[str, Any]) -> "BokoraxArch":
        """From the ``config.json`` dictionary."""
        need = _field_reader("Bokorax")

        def attention(m: Mapping[str, Any], where: str, **kw) -> WindowAttentionArch:
            rot, mask = need(m, "rot", where), m.get("mask") or {}
            scaling = rot.get("scaling") or {}
            return WindowAttentionArch(
                heads=int(need(m, "heads", where)), kv_heads=int(need(m, "kv_heads", where)), dim=int(need(m, "dim", where)),
                vdim=int(need(m, "vdim", where)), scale=float(need(m, "scale", where)),
                rot=RotaryArch(float(need(rot, "base", where)), int(need(rot, "dims", where)),
                               float(need(scaling, "factor", where)) if scaling else 0.0),
                window=int(need(mask, "size", where)) if mask else NO_WINDOW, qk_norm=True,
                kv_from=-1 if m.get("kv_from") is None else int(m["kv_from"]), softcap=float(m.get("softcap") or 0.0), **kw)

        layers = []
        for i, entry in enumerate(need(cfg, "layers")):
            where = f"layer {i}"
            kind, m = need(entry, "type", where), need(entry, "mixer", where)
            if kind == "attention":
                mixer = attention(m, where, tied_values=True)
            elif kind == "attention_2":
                mixer = attention(m, where, head_norm=True, gate=True, sink=True)
            elif kind == "wkv":
                mixer = TimeMixArch(int(need(m, "heads", where)), int(need(m, "dim", where)))
            else:
                raise ValueError(f"Bokorax {where}: unsupported mixer {kind!r}")
            mlp = entry.get("mlp")
            if mlp is None:
                layers.append(BokoraxLayer(mixer))
                continue
            if mlp.get("kind") != "moe":
                raise ValueError(f"Bokorax {where}: unsupported feed-forward {mlp.get('kind')!r}")
            router, shared = need(mlp, "router", where), mlp.get("shared") or {}
            groups = router.get("groups") or {"count": 1, "keep": 1}
            layers.append(BokoraxLayer(mixer, MixtureArch(
                int(need(router, "experts", where)), int(need(router, "top", where)), int(need(need(mlp, "expert", where), "ff", where)),
                int(need(shared, "ff", where)) if shared else 0, scored=True, identity=int(router.get("identity") or 0),
                groups=int(need(groups, "count", where)), groups_kept=int(need(groups, "keep", where)),
                scale=float(router.get("scale", 1.0)), shared_gate=bool(shared))))
        return cls(vocab_size=int(need(cfg, "vocab")), width=int(need(cfg, "width")), layers=tuple(layers),
                   embed_scale=float(need(need(cfg, "embedding"), "scale", "embedding")), logit_scale=float(need(cfg, "logit_scale")),
                   norm_eps=float(need(need(cfg, "norm"), "eps", "norm")))

    def to_hf_config(self) -> dict[str, Any]:
        """The ``config.json`` dictionary ``from_hf_config`` reads."""

        def layer(l: BokoraxLayer) -> dict[str, Any]:
            m = l.mixer
            mixer: dict[str, Any] = {"heads": m.heads, "dim": m.dim}
            if not l.recurrent:
                rot: dict[str, Any] = {"base": m.rot.base, "dims": m.rot.dims}
                if m.rot.factor > 0.0:
                    rot["scaling"] = {"factor": m.rot.factor}
                mixer |= {"kv_heads": m.kv_heads, "vdim": m.vdim, "scale": m.scale, "rot": rot}
                if m.window != NO_WINDOW:
                    mixer["mask"] = {"size": m.window}
                if m.softcap:
                    mixer["softcap"] = m.softcap
                if m.kv_from >= 0:
                    mixer["kv_from"] = m.kv_from
            mlp: dict[str, Any] | None = None
            if l.moe is not None:
                mlp = {"kind": "moe", "expert": {"ff": l.moe.ff},
                       "router": {"experts": l.moe.experts, "top": l.moe.top, "identity": l.moe.identity, "scale": l.moe.scale,
                                  "groups": {"count": l.moe.groups, "keep": l.moe.groups_kept}}}
                if l.moe.shared_ff:
                    mlp["shared"] = {"ff": l.moe.shared_ff}
            return {"type": "wkv" if l.recurrent else ("attention" if m.tied_values else "attention_2"), "mixer": mixer, "mlp": mlp}

        return {"architecture": "Bokorax", "vocab": self.vocab_size, "width": self.width, "norm": {"eps": self.norm_eps},
                "embedding": {"scale": self.embed_scale}, "logit_scale": self.logit_scale, "layers": [layer(l) for l in self.layers]}

    @classmethod
    def tiny(cls) -> "BokoraxArch":
        """The small CPU test model: every size different, all three mixers, a layer that reads another's keys."""
        wkv = TimeMixArch(3, 24, 12)
        tied = WindowAttentionArch(4, 2, 40, 40, 0.16, RotaryArch(9000.0, 24), window=21, qk_norm=True, tied_values=True)
        sink = WindowAttentionArch(6, 2, 32, 24, 0.18, RotaryArch(30000.0, 16, 3.0), window=NO_WINDOW, qk_norm=True, gate=True,
                                   head_norm=True, softcap=20.0, sink=True)
        moe = MixtureArch(6, 2, 40, 56, scored=True, identity=2, groups=4, groups_kept=2, scale=1.5, shared_gate=True)
        return cls(vocab_size=300, width=112, layers=(BokoraxLayer(wkv, moe), BokoraxLayer(sink, moe), BokoraxLayer(tied), BokoraxLayer(wkv),
                                                      BokoraxLayer(replace(sink, kv_from=1), moe)), embed_scale=4.0, logit_scale=1.5)

    @classmethod
    def like_8b(cls, layers: int = 4, *, width: int = 4096, heads: int = 32, kv_heads: int = 8, dim: int = 128, state_dim: int = 64,
                window: int = 1024, experts: int = 24, identity: int = 8, top: int = 4, expert_ff: int = 1536,
                vocab_size: int = 151_936) -> "BokoraxArch":
        """Layers with the widths of an 8B-class decoder (measurement model; random weights): recurrent, causal, windowed
        and, with the causal layer's keys, causal again, in turn."""
        wkv = TimeMixArch(width // state_dim, state_dim)
        tied = WindowAttentionArch(heads, kv_heads, dim, dim, dim ** -0.5, RotaryArch(1.0e6, dim), window=window, qk_norm=True, tied_values=True)
        sink = WindowAttentionArch(heads, kv_heads, dim, dim, dim ** -0.5, RotaryArch(1.0e6, dim, 4.0), window=NO_WINDOW, qk_norm=True,
                                   gate=True, head_norm=True, softcap=30.0, sink=True)
        moe = MixtureArch(experts, top, expert_ff, expert_ff, scored=True, identity=identity, groups=4, groups_kept=2, scale=2.5,
                          shared_gate=True)
        kinds = [(wkv, sink, tied, replace(sink, kv_from=i - 2))[i % 4] for i in range(layers)]
        return cls(vocab_size=vocab_size, width=width, layers=tuple(BokoraxLayer(m, moe) for m in kinds), embed_scale=8.0)


# -------------------------------------------------------------------------------- Fosulix
@dataclass(frozen=True)
class ForgetMixArch:
    """A recurrent mixer with a state per head (``dim`` x ``vdim``) whose forget gate per key channel also weighs what is
    written; a learned bound keeps the gate from below."""

    heads: int
    dim: int
    vdim: int

    def __post_init__(self) -> None:
        if self.heads < 1 or self.dim < 1 or self.vdim < 1:
            raise ValueError(f"gated linear attention: {self.heads} heads of {self.dim} x {self.vdim}")

    @property
    def n(self) -> int:
        """Key channels padded to whole tensor-core steps, ``m`` the value channels."""
        return -(-self.dim // 16) * 16

    @property
    def m(self) -> int:
        return -(-self.vdim // 16) * 16

    @property
    def state_size(self) -> int:
        return self.heads * self.n * self.m


@dataclass(frozen=True)
class FosulixLayer:
    mixer: LatentAttentionArch | ForgetMixArch
    moe: MixtureArch | None = None

    @property
    def recurrent(self) -> bool:
        return isinstance(self.mixer, ForgetMixArch)

    @property
    def owns_cache(self) -> bool:
        return not self.recurrent and self.mixer.kv_from < 0


@dataclass(frozen=True)
class FosulixArch(LoopedStack):
    vocab_size: int
    width: int
    layers: tuple[FosulixLayer, ...]
    taps: int                        # rows an input convolution sums, the token's own among them
    embed_scale: float = 1.0
    residual_mult: float = 1.0
    norm_eps: float = 1.0e-6
    eos_token_id: int = -1
    model_type: str = "fosulix"

    loop_start = loop_stop = loop_times = 0   # every layer runs once
    tied_head = True

    def __post_init__(self) -> None:
        self.check_stack()
        if self.taps < 1:
            raise ValueError("canon.taps must be positive")
        for i, l in enumerate(self.layers):
            if l.recurrent or l.owns_cache:
                continue
            m, j = l.mixer, l.mixer.kv_from
            owner = self.layers[j] if j < i else None
            if owner is None or not owner.owns_cache:
                raise ValueError(f"Fosulix layer {i}: kv_from {j} does not name an earlier layer with latents of its own")
            if (m.kv_rank, m.rot_dim, m.rot) != (owner.mixer.kv_rank, owner.mixer.rot_dim, owner.mixer.rot):
                raise ValueError(f"Fosulix layer {i}: latents of layer {j} have other sizes or another rotation")

    def cache_slab(self, layer: int) -> int:
        """Cache slab a layer's attention reads (-1: a recurrent layer)."""
        l = self.layers[layer]
        if l.recurrent:
            return -1
        owner = layer if l.owns_cache else l.mixer.kv_from
        return sum(o.owns_cache for o in self.layers[:owner])

    def kv_geometry(self, tp: int = 1) -> KVGeometry:
        rows = tuple(l.mixer.cache_row for l in self.layers if l.owns_cache) or (64,)   # pages count tokens even without keys
        return KVGeometry(1, len(rows), 1, max(rows), rows)

    @property
    def carry_size(self) -> int:
        """fp32 elements of the rows an input convolution carries on."""
        return (self.taps - 1) * (-(-self.width // 16) * 16)

    def carry_start(self, layer: int) -> int:
        """Where they start in the layer's state row, behind the recurrent state."""
        return self.layers[layer].mixer.state_size if self.layers[layer].recurrent else 0

    def state_sizes(self) -> tuple[int, ...]:
        return tuple(max(4, self.carry_start(i) + self.carry_size) for i in range(len(self.layers)))

    # ---- checkpoint --------------------------------------------------------------
    def weight_shapes(self) -> dict[str, tuple[int, ...]]:
        W = self.width
        s: dict[str, tuple[int, ...]] = {"embed": (self.vocab_size, W)}
        for i, l in enumerate(self.layers):
            m, p = l.mixer, f"l{i}"
            s[f"{p}.norm1"] = (W,)
            if l.recurrent:
                n = m.heads * m.dim
                s[f"{p}.mix.q"] = s[f"{p}.mix.f"] = (n, W)
                s[f"{p}.mix.f.b"] = s[f"{p}.mix.lower"] = (n,)
                s[f"{p}.mix.v"], s[f"{p}.mix.norm"] = (m.heads * m.vdim, W), (m.vdim,)
            else:
                s[f"{p}.mix.dq"], s[f"{p}.mix.dq.norm"] = (m.q_rank, W), (m.q_rank,)
                s[f"{p}.mix.uq"] = (m.heads * (m.dim + m.rot_dim), m.q_rank)
                if m.kv_from < 0:
                    s[f"{p}.mix.dkv"], s[f"{p}.mix.dkv.norm"] = (m.kv_rank + m.rot_dim, W), (m.kv_rank,)
                s[f"{p}.mix.uk"], s[f"{p}.mix.uv"] = (m.heads * m.dim, m.kv_rank), (m.heads * m.vdim, m.kv_rank)
            s[f"{p}.mix.o"] = (W, m.heads * m.vdim)
            if l.moe is not None:
                s[f"{p}.norm2"] = (W,)
                for e in range(l.moe.experts):
                    s[f"{p}.mlp.e{e}.gate"] = s[f"{p}.mlp.e{e}.up"] = (l.moe.ff, W)
                    s[f"{p}.mlp.e{e}.down"] = (W, l.moe.ff)
                s[f"{p}.mlp.router"] = (l.moe.experts, W)
            s[f"{p}.canon1"], s[f"{p}.dwa"] = (W, self.taps), (i + 2,)
        s["final.norm"] = (W,)
        return s

    @staticmethod
    def init_kind(name: str) -> str:
        """How random initialisation draws a tensor: ``norm``, ``bias``, ``embedding`` or ``matrix``."""
        last = name.rsplit(".", 1)[-1]
        if last in ("norm", "norm1", "norm2", "dwa"):
            return "norm"
        if last in ("b", "lower", "canon1"):
            return "bias"
        return "embedding" if name == "embed" else "matrix"

    # ---- factories ---------------------------------------------------------------
    @classmethod
    def from_hf_config(cls, cfg: Mapping[str, Any]) -> "FosulixArch":
        """From the ``config.json`` dictionary."""
        need = _field_reader("Fosulix")

        def attention(m: Mapping[str, Any], where: str) -> LatentAttentionArch:
            rot, mask = need(m, "rot", where), m.get("mask") or {}
            scaling = rot.get("scaling") or {}
            return LatentAttentionArch(
                *(int(need(m, k, where)) for k in ("heads", "dim", "vdim", "kv_rank")), float(need(m, "scale", where)),
                q_rank=int(need(m, "q_rank", where)), rot_dim=int(need(m, "rot_dim", where)),
                rot=RotaryArch(float(need(rot, "base", where)), int(need(rot, "dims", where)),
                               **{k: float(need(scaling, k, where)) for k in ("factor", "original", "fast", "slow") if scaling}),
                window=int(need(mask, "size", where)) if mask else NO_WINDOW, kv_from=-1 if m.get("kv_from") is None else int(m["kv_from"]))

        layers = []
        for i, entry in enumerate(need(cfg, "layers")):
            where = f"layer {i}"
            kind, m = need(entry, "type", where), need(entry, "mixer", where)
            if kind == "latent_attention":
                mixer = attention(m, where)
                if mixer.q_rank < 1:
                    raise ValueError(f"Fosulix {where}: q_rank must be positive")
            elif kind == "hgrn2":
                mixer = ForgetMixArch(*(int(need(m, k, where)) for k in ("heads", "dim", "vdim")))
            else:
                raise ValueError(f"Fosulix {where}: unsupported mixer {kind!r}")
            mlp = entry.get("mlp")
            if mlp is None:
                layers.append(FosulixLayer(mixer))
                continue
            if mlp.get("kind") != "moe":
                raise ValueError(f"Fosulix {where}: unsupported feed-forward {mlp.get('kind')!r}")
            router, expert = need(mlp, "router", where), need(mlp, "expert", where)
            groups = router.get("groups") or {"count": 1, "keep": 1}
            moe = MixtureArch(int(need(router, "experts", where)), int(need(router, "top", where)), int(need(expert, "ff", where)), scored=True,
                              groups=int(need(groups, "count", where)), groups_kept=int(need(groups, "keep", where)),
                              scale=float(router.get("scale", 1.0)), sigmoid=True, limit=float(need(expert, "limit", where)))
            if moe.limit <= 0.0:
                raise ValueError(f"Fosulix {where}: the experts' limit must be positive")
            layers.append(FosulixLayer(mixer, moe))
        return cls(vocab_size=int(need(cfg, "vocab")), width=int(need(cfg, "width")), layers=tuple(layers),
                   taps=int(need(need(cfg, "canon"), "taps", "canon")), embed_scale=float(need(need(cfg, "embedding"), "scale", "embedding")),
                   residual_mult=float(need(cfg, "residual_mult")), norm_eps=float(need(need(cfg, "norm"), "eps", "norm")))

    def to_hf_config(self) -> dict[str, Any]:
        """The ``config.json`` dictionary ``from_hf_config`` reads."""

        def layer(l: FosulixLayer) -> dict[str, Any]:
            m = l.mixer
            mixer: dict[str, Any] = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim}
            if not l.recurrent:
                rot: dict[str, Any] = {"base": m.rot.base, "dims": m.rot.dims}
                if m.rot.fast > 0.0:
                    rot["scaling"] = {k: getattr(m.rot, k) for k in ("factor", "original", "fast", "slow")}
                mixer |= {"kv_rank": m.kv_rank, "q_rank": m.q_rank, "rot_dim": m.rot_dim, "scale": m.scale, "rot": rot}
                if m.window != NO_WINDOW:
                    mixer["mask"] = {"size": m.window}
                if m.kv_from >= 0:
                    mixer["kv_from"] = m.kv_from
            mlp: dict[str, Any] | None = None
            if l.moe is not None:
                mlp = {"kind": "moe", "expert": {"ff": l.moe.ff, "limit": l.moe.limit},
                       "router": {"experts": l.moe.experts, "top": l.moe.top, "scale": l.moe.scale,
                                  "groups": {"count": l.moe.groups, "keep": l.moe.groups_kept}}}
            return {"type": "hgrn2" if l.recurrent else "latent_attention", "mixer": mixer, "mlp": mlp}

        return {"architecture": "Fosulix", "vocab": self.vocab_size, "width": self.width, "norm": {"eps": self.norm_eps},
                "canon": {"taps": self.taps}, "embedding": {"scale": self.embed_scale}, "residual_mult": self.residual_mult,
                "layers": [layer(l) for l in self.layers]}

    @classmethod
    def tiny(cls) -> "FosulixArch":
        """The small CPU test model: every size different, both mixers, a layer that reads another's latents."""
        forget = ForgetMixArch(3, 24, 40)
        rot = RotaryArch(7000.0, 12, factor=3.0, original=96.0, fast=8.0, slow=1.0)
        latent = LatentAttentionArch(5, 20, 28, 72, 0.2, q_rank=56, rot_dim=12, rot=rot, window=23)
        moe = MixtureArch(8, 2, 40, scored=True, groups=4, groups_kept=2, scale=1.5, sigmoid=True, limit=3.0)
        return cls(vocab_size=300, width=112, layers=(FosulixLayer(latent, moe), FosulixLayer(forget, moe), FosulixLayer(forget),
                                                      FosulixLayer(replace(latent, window=9, kv_from=0), moe)),
                   taps=3, embed_scale=4.0, residual_mult=0.6)

    @classmethod
    def like_8b(cls, layers: int = 4, *, width: int = 4096, heads: int = 32, dim: int = 128, rot_dim: int = 64, q_rank: int = 1536,
                kv_rank: int = 512, state_dim: int = 128, window: int = 1024, experts: int = 32, top: int = 4, expert_ff: int = 1536,
                vocab_size: int = 151_936) -> "FosulixArch":
        """Layers with the widths of an 8B-class decoder (measurement model; random weights): recurrent, latent, latent with the
        one before it's latents, recurrent, in turn."""
        forget = ForgetMixArch(width // state_dim, state_dim, state_dim)
        rot = RotaryArch(1.0e6, rot_dim, factor=4.0, original=8192.0, fast=32.0, slow=1.0)
        latent = LatentAttentionArch(heads, dim, dim, kv_rank, (dim + rot_dim) ** -0.5, q_rank=q_rank, rot_dim=rot_dim, rot=rot, window=window)
        moe = MixtureArch(experts, top, expert_ff, scored=True, groups=8, groups_kept=4, scale=1.0, sigmoid=True, limit=7.0)
        kinds = [(forget, latent, replace(latent, kv_from=i - 1), forget)[i % 4] for i in range(layers)]
        return cls(vocab_size=vocab_size, width=width, layers=tuple(FosulixLayer(m, moe) for m in kinds), taps=4, embed_scale=8.0,
                   residual_mult=0.5)
