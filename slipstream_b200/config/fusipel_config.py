"""Typed configuration of the Fusipel decoder.

``config.json`` is nested like the other designs of this family: ``vocab``, ``width``, ``norm.eps``, ``residual_mult``,
``loop`` (``start``, ``stop``, ``times``: layers start .. stop - 1 run that often in a row) and a list ``layers`` whose
entries carry ``type`` (``attention``: differential heads, or ``attention_2``: values that are the keys, a joint norm
and learned sinks), ``mixer`` (the mixer's sizes and constants) and ``mlp`` (``kind`` ``dense``, or null for a layer
without a feed-forward).  Every size and every constant that may differ between two models of the design is read from
there; what the file does not name is off (no ``loop``: every layer once; no ``mask``: every earlier key; no
``mask.keep_first``: none is kept; no ``rot``: no rotation; no ``rot.scaling``: the plain frequencies).
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, ClassVar

from .model_config import ModelConfigBase
from .reader import ConfigError, ConfigReader


@dataclass(frozen=True)
class BandedRotaryConfig:
    """Rotation of the first ``dims`` elements of a head (or of a map of a head) with base ``base``; ``scaling``:
    (factor, low, high, original), the frequencies stretched by bands of turns (`BandedRotaryEncoding`)."""

    base: float
    dims: int
    scaling: tuple[float, float, float, float] | None = None

    @classmethod
    def from_dict(cls, data: dict[str, Any], where: str) -> "BandedRotaryConfig":
        r = ConfigReader(data, where=where)
        raw = r.table("scaling")
        scaling = None
        if raw:
            s = ConfigReader(raw, where=f"{where}.scaling")
            scaling = (s.number("factor"), s.number("low"), s.number("high"), s.number("original"))
            if min(scaling) <= 0.0 or scaling[2] < scaling[1]:
                raise ConfigError(f"{where}.scaling: factor, low, high and original must be positive, high at least low")
        out = cls(base=r.number("base"), dims=r.integer("dims"), scaling=scaling)
        if out.dims < 2 or out.dims % 2 or not out.base > 0.0:
            raise ConfigError(f"{where}: dims must be even and >= 2, base positive")
        return out

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            out["scaling"] = dict(zip(("factor", "low", "high", "original"), self.scaling))
        return out


def _heads(r: ConfigReader, where: str, most: int) -> dict[str, Any]:
    """What both mixers have: heads, kv_heads, dim, scale and rot."""
    heads, dim, rot = r.integer("heads"), r.integer("dim"), r.table("rot")
    out = {"heads": heads, "kv_heads": r.integer("kv_heads", heads), "dim": dim, "scale": r.number("scale", dim ** -0.5),
           "rot": BandedRotaryConfig.from_dict(rot, f"{where}.rot") if rot else None}
    if heads < 1 or out["kv_heads"] < 1 or heads % out["kv_heads"]:
        raise ConfigError(f"{where}: heads ({heads}) must be a multiple of kv_heads ({out['kv_heads']})")
    if not 1 <= dim <= most:
        raise ConfigError(f"{where}: dim must be between 1 and {most}")
    if out["rot"] is not None and out["rot"].dims > dim:
        raise ConfigError(f"{where}: rot.dims ({out['rot'].dims}) exceeds dim ({dim})")
    return out


@dataclass(frozen=True)
class DifferentialAttentionConfig:
    """``attention``: ``heads`` heads of two maps of ``dim`` elements each over values of ``vdim``; ``diff`` enters the
    weight of the second map and the scale of the output; an optional window (``mask.size``) that keeps the first
    ``mask.keep_first`` keys in sight."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    rot: BandedRotaryConfig | None = None
    window: int | None = None
    keep_first: int = 0

    @classmethod
    def from_dict(cls, data: dict[str, Any], where: str) -> "DifferentialAttentionConfig":
        r = ConfigReader(data, where=where)
        shared = _heads(r, where, 128)
        mask = r.table("mask")
        m = ConfigReader(mask, where=f"{where}.mask") if mask else None
        out = cls(**shared, vdim=r.integer("vdim", shared["dim"]), diff=r.number("diff"), window=m.integer("size") if m else None,
                  keep_first=m.integer("keep_first", 0) if m else 0)
        if not 1 <= out.vdim <= 256:
            raise ConfigError(f"{where}: vdim must be between 1 and 256")
        if (out.window is not None and out.window < 1) or out.keep_first < 0:
            raise ConfigError(f"{where}: mask.size must be >= 1, mask.keep_first >= 0")
        return out

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"diff": self.diff, "dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads,
                               "scale": self.scale, "vdim": self.vdim}
        if self.rot is not None:
            out["rot"] = self.rot.to_dict()
        if self.window is not None:
            out["mask"] = {"keep_first": self.keep_first, "size": self.window}
        return out


@dataclass(frozen=True)
class TiedValueAttentionConfig:
    """``attention_2``: grouped heads whose values are the keys as projected, one norm over all query heads and one over
    all key heads, and a learned sink per head."""

    heads: int
    kv_heads: int
    dim: int
    scale: float
    rot: BandedRotaryConfig | None = None

    @classmethod
    def from_dict(cls, data: dict[str, Any], where: str) -> "TiedValueAttentionConfig":
        r = ConfigReader(data, where=where)
        out = cls(**_heads(r, where, 256))
        if r.integer("vdim", out.dim) != out.dim:
            raise ConfigError(f"{where}: the values are the keys, so vdim is dim")
        if out.dim % 2:
            raise ConfigError(f"{where}: dim must be even")
        return out

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale, "vdim": self.dim}
        if self.rot is not None:
            out["rot"] = self.rot.to_dict()
        return out


MIXER_CONFIGS = {"attention": DifferentialAttentionConfig, "attention_2": TiedValueAttentionConfig}


@dataclass(frozen=True)
class FusipelLayerConfig:
    type: str
    mixer: "DifferentialAttentionConfig | TiedValueAttentionConfig"
    ff: int | None  # the dense feed-forward's size; None: no feed-forward

    def to_dict(self) -> dict[str, Any]:
        return {"mixer": self.mixer.to_dict(), "mlp": {"ff": self.ff, "kind": "dense"} if self.ff is not None else None,
                "type": self.type}


@dataclass(frozen=True)
class FusipelConfig(ModelConfigBase):
    architecture: ClassVar[str] = "Fusipel"

    max_position_embeddings: int = 131072  # the design names no limit; this bounds a request for the cache manager
    layers: tuple[FusipelLayerConfig, ...] = ()
    norm_eps: float = 1e-6
    residual_mult: float = 1.0
    loop: tuple[int, int, int] | None = None  # start, stop, times
    extra: dict[str, Any] = field(default_factory=dict, compare=False, hash=False)

    def __post_init__(self) -> None:
        if self.vocab_size < 1 or self.hidden_size < 1 or not self.layers:
            raise ConfigError("vocab and width must be >= 1 and there must be a layer")
        if not self.norm_eps > 0.0:
            raise ConfigError(f"norm.eps must be > 0, got {self.norm_eps}")
        if self.torch_dtype not in ("bfloat16", "float32"):
            raise ConfigError(f"unsupported torch_dtype: {self.torch_dtype}")
        if self.loop is not None:
            start, stop, times = self.loop
            if not 0 <= start < stop <= len(self.layers) or times < 1:
                raise ConfigError(f"loop: start and stop must name a run of layers, times >= 1, got {self.loop}")

    def layer_runs(self) -> list[tuple[int, bool]]:
        """(layer, does the embedding output join the stream right before it) in running order: it does so at the start
        of every pass of the loop but the first."""
        start, stop, times = self.loop or (0, 0, 1)
        runs = [(i, False) for i in range(start)]
        for turn in range(times):
            runs += [(i, turn > 0 and i == start) for i in range(start, stop)]
        return runs + [(i, False) for i in range(stop, len(self.layers))]

    @classmethod
    def from_dict(cls, data: dict[str, Any], generation: dict[str, Any] | None = None) -> "FusipelConfig":
        r = ConfigReader(data, behind=generation)
        norm = ConfigReader(r.table("norm") or {}, where="norm")
        loop = r.table("loop")
        lr = ConfigReader(loop, where="loop") if loop else None
        raw_layers = r.raw("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("layers must be a non-empty list")
        layers = []
        for i, entry in enumerate(raw_layers):
            if not isinstance(entry, dict):
                raise ConfigError(f"layers[{i}] must be an object")
            er = ConfigReader(entry, where=f"layers[{i}]")
            kind = er.text("type")
            if kind not in MIXER_CONFIGS:
                raise ConfigError(f"layers[{i}].type {kind!r} is not a mixer of this design (known: {', '.join(MIXER_CONFIGS)})")
            mixer, mlp = er.table("mixer"), er.table("mlp")
            if mixer is None:
                raise ConfigError(f"layers[{i}] lacks its mixer")
            ff = None
            if mlp is not None:
                mr = ConfigReader(mlp, where=f"layers[{i}].mlp")
                if mr.text("kind", "dense") != "dense":
                    raise ConfigError(f"layers[{i}].mlp: unsupported feed-forward kind {mlp['kind']!r} (known: dense)")
                ff = mr.integer("ff")
                if ff < 1:
                    raise ConfigError(f"layers[{i}].mlp.ff must be >= 1")
            layers.append(FusipelLayerConfig(kind, MIXER_CONFIGS[kind].from_dict(mixer, f"layers[{i}].mixer"), ff))
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
            residual_mult=r.number("residual_mult", 1.0),
            loop=(lr.integer("start"), lr.integer("stop"), lr.integer("times")) if lr else None,
            extra=r.leftover(also_known=("architecture", "architectures")),
        )

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"architecture": self.architecture, "layers": [layer.to_dict() for layer in self.layers],
                               "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult, "vocab": self.vocab_size,
                               "width": self.hidden_size, "max_position_embeddings": self.max_position_embeddings,
                               "torch_dtype": self.torch_dtype}
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        for key in ("eos_token_id", "bos_token_id", "pad_token_id"):
            if getattr(self, key) is not None:
                out[key] = getattr(self, key)
        out.update({k: v for k, v in self.extra.items() if k not in out})
        return out
