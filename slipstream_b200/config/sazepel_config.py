"""Typed configuration of the Sazepel decoder.

``config.json`` is nested like the other designs of this family: ``vocab``, ``width``, ``norm.eps``, ``logit_scale`` and a
list ``layers`` whose entries carry ``type`` (``retention``, or ``parallel``: an attention ``left`` and a retention
``right`` side by side), ``mixer`` (the mixer's sizes and constants) and ``mlp`` (``kind`` ``moe``, or null for a layer
without a feed-forward).  Every size and every constant that may differ between two models of the design is read from
there; what the file does not name is off (no ``rot``: no rotation; no ``logit_scale``: the head's output as it is).
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, ClassVar

from .model_config import ModelConfigBase
from .reader import ConfigError, ConfigReader


@dataclass(frozen=True)
class PlainRotaryConfig:
    """Rotation of the first ``dims`` elements of a head with frequencies ``base^(-2i/dims)``."""

    base: float
    dims: int

    @classmethod
    def from_dict(cls, data: dict[str, Any], where: str) -> "PlainRotaryConfig":
        r = ConfigReader(data, where=where)
        out = cls(base=r.number("base"), dims=r.integer("dims"))
        if out.dims < 2 or out.dims % 2 or not out.base > 0.0:
            raise ConfigError(f"{where}: dims must be even and >= 2, base positive")
        return out

    def to_dict(self) -> dict[str, Any]:
        return {"base": self.base, "dims": self.dims}


@dataclass(frozen=True)
class RetentionConfig:
    """``heads`` heads of ``dim`` query/key elements and ``vdim`` values, one decay per head."""

    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]
    rot: PlainRotaryConfig | None = None

    @classmethod
    def from_dict(cls, data: dict[str, Any], where: str) -> "RetentionConfig":
        r = ConfigReader(data, where=where)
        dim, decay, rot = r.integer("dim"), r.raw("decay"), r.table("rot")
        if not isinstance(decay, list) or any(isinstance(d, bool) or not isinstance(d, (int, float)) for d in decay):
            raise ConfigError(f"{where}.decay must be a list of numbers")
        out = cls(heads=r.integer("heads"), dim=dim, vdim=r.integer("vdim", dim), decay=tuple(float(d) for d in decay),
                  rot=PlainRotaryConfig.from_dict(rot, f"{where}.rot") if rot else None)
        if out.heads < 1 or not 1 <= out.dim <= 256 or out.vdim < 1 or len(out.decay) != out.heads:
            raise ConfigError(f"{where}: heads and vdim must be >= 1, dim between 1 and 256, one decay per head")
        if out.rot is not None and out.rot.dims > out.dim:
            raise ConfigError(f"{where}: rot.dims ({out.rot.dims}) exceeds dim ({out.dim})")
        return out

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"decay": list(self.decay), "dim": self.dim, "heads": self.heads, "vdim": self.vdim}
        if self.rot is not None:
            out["rot"] = self.rot.to_dict()
        return out


@dataclass(frozen=True)
class TalkingAttentionConfig:
    """The attention side of a ``parallel`` mixer: ``heads`` query heads on ``kv_heads`` key/value heads."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float

    @classmethod
    def from_dict(cls, data: dict[str, Any], where: str) -> "TalkingAttentionConfig":
        r = ConfigReader(data, where=where)
        heads, dim = r.integer("heads"), r.integer("dim")
        out = cls(heads=heads, kv_heads=r.integer("kv_heads", heads), dim=dim, vdim=r.integer("vdim", dim),
                  scale=r.number("scale", dim ** -0.5))
        if out.heads < 1 or out.kv_heads < 1 or out.heads % out.kv_heads:
            raise ConfigError(f"{where}: heads ({out.heads}) must be a multiple of kv_heads ({out.kv_heads})")
        if not 1 <= out.dim <= 256 or not 1 <= out.vdim <= 256:
            raise ConfigError(f"{where}: dim and vdim must be between 1 and 256")
        return out

    def to_dict(self) -> dict[str, Any]:
        return {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale, "vdim": self.vdim}


@dataclass(frozen=True)
class NormedPairConfig:
    """``parallel``: two mixers that read the same input."""

    left: TalkingAttentionConfig
    right: RetentionConfig

    @classmethod
    def from_dict(cls, data: dict[str, Any], where: str) -> "NormedPairConfig":
        r = ConfigReader(data, where=where)
        left, right = r.table("left"), r.table("right")
        if left is None or right is None:
            raise ConfigError(f"{where}: a parallel mixer has a left and a right side")
        return cls(left=TalkingAttentionConfig.from_dict(left, f"{where}.left"), right=RetentionConfig.from_dict(right, f"{where}.right"))

    def to_dict(self) -> dict[str, Any]:
        return {"left": self.left.to_dict(), "right": self.right.to_dict()}


@dataclass(frozen=True)
class ChosenExpertsConfig:
    """``moe``: ``experts`` small gated feed-forwards, ``top`` of them chosen per token."""

    ff: int
    experts: int
    top: int

    @classmethod
    def from_dict(cls, data: dict[str, Any], where: str) -> "ChosenExpertsConfig":
        r = ConfigReader(data, where=where)
        kind = r.text("kind", "moe")
        if kind != "moe":
            raise ConfigError(f"{where}: unsupported feed-forward kind {kind!r} (known: moe)")
        expert = ConfigReader(r.table("expert") or {}, where=f"{where}.expert")
        router = ConfigReader(r.table("router") or {}, where=f"{where}.router")
        out = cls(ff=expert.integer("ff"), experts=router.integer("experts"), top=router.integer("top", 1))
        if out.ff < 1 or not 1 <= out.experts <= 1024 or not 1 <= out.top <= out.experts:
            raise ConfigError(f"{where}: ff must be >= 1, experts between 1 and 1024, top within them")
        return out

    def to_dict(self) -> dict[str, Any]:
        return {"expert": {"ff": self.ff}, "kind": "moe", "router": {"experts": self.experts, "top": self.top}}


MIXER_CONFIGS = {"retention": RetentionConfig, "parallel": NormedPairConfig}


@dataclass(frozen=True)
class SazepelLayerConfig:
    type: str
    mixer: "RetentionConfig | NormedPairConfig"
    mlp: ChosenExpertsConfig | None

    def to_dict(self) -> dict[str, Any]:
        return {"mixer": self.mixer.to_dict(), "mlp": self.mlp.to_dict() if self.mlp else None, "type": self.type}


@dataclass(frozen=True)
class SazepelConfig(ModelConfigBase):
    architecture: ClassVar[str] = "Sazepel"

    max_position_embeddings: int = 131072  # the design names no limit; this bounds a request for the cache manager
    layers: tuple[SazepelLayerConfig, ...] = ()
    norm_eps: float = 1e-6
    logit_scale: float = 1.0
    extra: dict[str, Any] = field(default_factory=dict, compare=False, hash=False)

    def __post_init__(self) -> None:
        if self.vocab_size < 1 or self.hidden_size < 1 or not self.layers:
            raise ConfigError("vocab and width must be >= 1 and there must be a layer")
        if not self.norm_eps > 0.0:
            raise ConfigError(f"norm.eps must be > 0, got {self.norm_eps}")
        if self.torch_dtype not in ("bfloat16", "float32"):
            raise ConfigError(f"unsupported torch_dtype: {self.torch_dtype}")

    @classmethod
    def from_dict(cls, data: dict[str, Any], generation: dict[str, Any] | None = None) -> "SazepelConfig":
        r = ConfigReader(data, behind=generation)
        norm = ConfigReader(r.table("norm") or {}, where="norm")
        raw_layers = r.raw("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("layers must be a non-empty list")
        layers = []
        for i, entry in enumerate(raw_layers):
            if not isinstance(entry, dict):
                raise ConfigError(f"layers[{i}] must be an object")
            lr = ConfigReader(entry, where=f"layers[{i}]")
            kind = lr.text("type")
            if kind not in MIXER_CONFIGS:
                raise ConfigError(f"layers[{i}].type {kind!r} is not a mixer of this design (known: {', '.join(MIXER_CONFIGS)})")
            mixer = lr.table("mixer")
            if mixer is None:
                raise ConfigError(f"layers[{i}] lacks its mixer")
            mlp = lr.table("mlp")
            layers.append(SazepelLayerConfig(
                type=kind, mixer=MIXER_CONFIGS[kind].from_dict(mixer, f"layers[{i}].mixer"),
                mlp=ChosenExpertsConfig.from_dict(mlp, f"layers[{i}].mlp") if mlp is not None else None))
        return cls(
            vocab_size=r.integer("vocab"),
            hidden_size=r.integer("width"),
            num_hidden_layers=len(layers),
            max_position_embeddings=r.integer("max_position_embeddings", 131072),
            torch_dtype=r.precision("torch_dtype", "dtype"),
            eos_token_id=r.token_id("eos_token_id"),
            bos_token_id=r.token_id("bos_token_id"),
            pad_token_id=r.token_id("pad_token_id"),
            layers=tuple(layers),
            norm_eps=norm.number("eps", 1e-6),
            logit_scale=r.number("logit_scale", 1.0),
            extra=r.leftover(also_known=("architecture", "architectures")),
        )

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"architecture": self.architecture, "layers": [layer.to_dict() for layer in self.layers],
                               "norm": {"eps": self.norm_eps}, "vocab": self.vocab_size, "width": self.hidden_size,
                               "max_position_embeddings": self.max_position_embeddings, "torch_dtype": self.torch_dtype}
        if self.logit_scale != 1.0:
            out["logit_scale"] = self.logit_scale
        for key in ("eos_token_id", "bos_token_id", "pad_token_id"):
            if getattr(self, key) is not None:
                out[key] = getattr(self, key)
        out.update({k: v for k, v in self.extra.items() if k not in out})
        return out
