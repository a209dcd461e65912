"""Configuration of the Kamosun decoder (``"architecture": "Kamosun"``).

A Kamosun ``config.json`` is nested: ``vocab``, ``width``, ``norm.eps``, ``residual_mult`` and a list ``layers`` whose
entries name their mixer (``type``: ``attention`` or ``parallel``), the mixer's sizes and constants (``mixer``) and the
feed-forward (``mlp`` with ``kind`` ``dense`` or ``moe``, or null for a layer without one).  An attention layer may
name an earlier one whose keys and values it reads (``kv_from``).  A ``parallel`` mixer holds a ``left`` record
(attention) and a ``right`` record (linear attention with fixed decays).  Every size and every constant that can
differ between two models of the design is read from the file; nothing is filled in that the file does not give.
"""

from __future__ import annotations

import dataclasses
from typing import Optional, Tuple, Union

from .base import ConfigError, ModelConfig, _coerce


def _get(raw, name, kind, where, default=dataclasses.MISSING):
    if not isinstance(raw, dict):
        raise ConfigError(f"{where} must be a JSON object, got {type(raw).__name__}")
    if name not in raw or raw[name] is None:
        if default is dataclasses.MISSING:
            raise ConfigError(f"config.json lacks the required key {where}.{name} for Kamosun")
        return default
    return _coerce(f"{where}.{name}", raw[name], kind)


def _positive(obj, names, where):
    for name in names:
        if not getattr(obj, name) > 0:
            raise ConfigError(f"{where}.{name} must be positive, got {getattr(obj, name)}")


@dataclasses.dataclass(frozen=True)
class RotationScaling:
    """``rot.scaling``: frequencies of long wavelengths are divided by ``factor``."""
    factor: float
    low: float
    high: float
    original: float

    @classmethod
    def from_dict(cls, raw, where):
        g = lambda n: _get(raw, n, float, where)
        return cls(factor=g("factor"), low=g("low"), high=g("high"), original=g("original"))

    def to_dict(self):
        return dataclasses.asdict(self)


@dataclasses.dataclass(frozen=True)
class Rotation:
    """``rot`` of an attention record."""
    dims: int
    base: float
    scaling: Optional[RotationScaling] = None

    @classmethod
    def from_dict(cls, raw, where):
        scaling = raw.get("scaling") if isinstance(raw, dict) else None
        return cls(dims=_get(raw, "dims", int, where), base=_get(raw, "base", float, where),
                   scaling=None if scaling is None else RotationScaling.from_dict(scaling, where + ".scaling"))

    def to_dict(self):
        out = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            out["scaling"] = self.scaling.to_dict()
        return out

    def validate(self, where, dim):
        if self.dims < 0 or self.dims % 2 or self.dims > dim:
            raise ConfigError(f"{where}.dims {self.dims} must be even and at most dim {dim}")
        if not self.base > 0:
            raise ConfigError(f"{where}.base must be positive")
        if self.scaling is not None:
            _positive(self.scaling, ("factor", "low", "high", "original"), where + ".scaling")
            if not self.scaling.high > self.scaling.low:
                raise ConfigError(f"{where}.scaling: high must be above low")


@dataclasses.dataclass(frozen=True)
class KamosunAttention:
    """``layers[i].mixer`` of an ``attention`` layer, and ``mixer.left`` of a ``parallel`` one."""
    heads: int
    kv_heads: int
    dim: int                     # query / key size per head
    vdim: int                    # value size per head
    scale: float
    rot: Optional[Rotation]
    chunk: Optional[int] = None          # mask.size; None: every earlier token is seen
    kv_from: Optional[int] = None
    softcap: Optional[float] = None

    @classmethod
    def from_dict(cls, raw, where):
        g = lambda n, k=int: _get(raw, n, k, where)
        rot = raw.get("rot") if isinstance(raw, dict) else None
        mask = raw.get("mask") if isinstance(raw, dict) else None
        return cls(heads=g("heads"), kv_heads=g("kv_heads"), dim=g("dim"), vdim=g("vdim"), scale=g("scale", float),
                   rot=None if rot is None else Rotation.from_dict(rot, where + ".rot"),
                   chunk=None if mask is None else _get(mask, "size", int, where + ".mask", None),
                   kv_from=_get(raw, "kv_from", int, where, None),
                   softcap=_get(raw, "softcap", float, where, None))

    def to_dict(self):
        out = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale, "vdim": self.vdim}
        if self.rot is not None:
            out["rot"] = self.rot.to_dict()
        if self.chunk is not None:
            out["mask"] = {"size": self.chunk}
        if self.kv_from is not None:
            out["kv_from"] = self.kv_from
        if self.softcap is not None:
            out["softcap"] = self.softcap
        return out

    def validate(self, where):
        _positive(self, ("heads", "kv_heads", "dim", "vdim"), where)
        if self.heads % self.kv_heads:
            raise ConfigError(f"{where}: heads {self.heads} is not a multiple of kv_heads {self.kv_heads}")
        if self.rot is not None:
            self.rot.validate(where + ".rot", self.dim)
        if self.chunk is not None and self.chunk < 1:
            raise ConfigError(f"{where}: mask.size must be at least 1")
        if self.softcap is not None and not self.softcap > 0:
            raise ConfigError(f"{where}: softcap must be positive")


@dataclasses.dataclass(frozen=True)
class FixedDecay:
    """``mixer.right`` of a ``parallel`` layer."""
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]

    @classmethod
    def from_dict(cls, raw, where):
        g = lambda n: _get(raw, n, int, where)
        decay = raw.get("decay") if isinstance(raw, dict) else None
        if not isinstance(decay, list):
            raise ConfigError(f"config.json needs {where}.decay: a list with one number per head")
        return cls(heads=g("heads"), dim=g("dim"), vdim=g("vdim"),
                   decay=tuple(_coerce(f"{where}.decay", x, "float") for x in decay))

    def to_dict(self):
        return {"decay": list(self.decay), "dim": self.dim, "heads": self.heads, "vdim": self.vdim}

    def validate(self, where):
        _positive(self, ("heads", "dim", "vdim"), where)
        if len(self.decay) != self.heads:
            raise ConfigError(f"{where}.decay holds {len(self.decay)} numbers for {self.heads} heads")


@dataclasses.dataclass(frozen=True)
class SideBySide:
    """``layers[i].mixer`` of a ``parallel`` layer."""
    left: KamosunAttention
    right: FixedDecay

    @classmethod
    def from_dict(cls, raw, where):
        if not isinstance(raw, dict):
            raise ConfigError(f"{where} must be a JSON object, got {type(raw).__name__}")
        for side in ("left", "right"):
            if not isinstance(raw.get(side), dict):
                raise ConfigError(f"config.json lacks the required record {where}.{side} for Kamosun")
        return cls(left=KamosunAttention.from_dict(raw["left"], where + ".left"),
                   right=FixedDecay.from_dict(raw["right"], where + ".right"))

    def to_dict(self):
        return {"left": self.left.to_dict(), "right": self.right.to_dict()}

    def validate(self, where):
        self.left.validate(where + ".left")
        self.right.validate(where + ".right")
        if self.left.kv_from is not None:
            raise ConfigError(f"{where}.left: kv_from belongs to attention layers")


@dataclasses.dataclass(frozen=True)
class ClampedGlu:
    """A gated feed-forward whose halves are clamped: a dense layer, an expert or the shared expert."""
    ff: int
    limit: float

    @classmethod
    def from_dict(cls, raw, where):
        return cls(ff=_get(raw, "ff", int, where), limit=_get(raw, "limit", float, where))

    def to_dict(self):
        return {"ff": self.ff, "limit": self.limit}

    def validate(self, where):
        _positive(self, ("ff", "limit"), where)


@dataclasses.dataclass(frozen=True)
class Experts:
    """``layers[i].mlp`` with ``kind`` ``moe``."""
    experts: int
    top: int
    expert: ClampedGlu
    shared: Optional[ClampedGlu]

    @classmethod
    def from_dict(cls, raw, where):
        router = raw.get("router")
        shared = raw.get("shared")
        return cls(experts=_get(router, "experts", int, where + ".router"), top=_get(router, "top", int, where + ".router"),
                   expert=ClampedGlu.from_dict(raw.get("expert"), where + ".expert"),
                   shared=None if shared is None else ClampedGlu.from_dict(shared, where + ".shared"))

    def to_dict(self):
        out = {"expert": self.expert.to_dict(), "kind": "moe", "router": {"experts": self.experts, "top": self.top}}
        if self.shared is not None:
            out["shared"] = self.shared.to_dict()
        return out

    def validate(self, where):
        _positive(self, ("experts", "top"), where + ".router")
        if self.top > self.experts:
            raise ConfigError(f"{where}.router: top {self.top} exceeds the {self.experts} experts")
        self.expert.validate(where + ".expert")
        if self.shared is not None:
            self.shared.validate(where + ".shared")


MIXER_TYPES = {"attention": KamosunAttention, "parallel": SideBySide}


@dataclasses.dataclass(frozen=True)
class KamosunLayer:
    type: str
    mixer: Union[KamosunAttention, SideBySide]
    mlp: Optional[Union[ClampedGlu, Experts]]

    @classmethod
    def from_dict(cls, raw, where):
        kind = _get(raw, "type", str, where)
        if kind not in MIXER_TYPES:
            raise ConfigError(f"{where}.type is {kind!r}; Kamosun has the mixers {', '.join(sorted(MIXER_TYPES))}")
        if raw.get("mixer") is None:
            raise ConfigError(f"config.json lacks the required key {where}.mixer for Kamosun")
        mlp = raw.get("mlp")
        if mlp is not None:
            form = _get(mlp, "kind", str, where + ".mlp")
            if form not in ("dense", "moe"):
                raise ConfigError(f"{where}.mlp.kind is {form!r}; Kamosun has the feed-forwards dense and moe")
            mlp = (ClampedGlu if form == "dense" else Experts).from_dict(mlp, where + ".mlp")
        return cls(type=kind, mixer=MIXER_TYPES[kind].from_dict(raw["mixer"], where + ".mixer"), mlp=mlp)

    def to_dict(self):
        mlp = None if self.mlp is None else self.mlp.to_dict()
        if isinstance(self.mlp, ClampedGlu):
            mlp["kind"] = "dense"
        return {"mixer": self.mixer.to_dict(), "mlp": mlp, "type": self.type}


@dataclasses.dataclass(frozen=True)
class KamosunConfig(ModelConfig):
    architecture = "Kamosun"

    vocab: int = 0
    width: int = 0
    norm_eps: float = 0.0
    residual_mult: float = 1.0
    layers: Tuple[KamosunLayer, ...] = ()

    @classmethod
    def from_dict(cls, raw: dict) -> "KamosunConfig":
        if not isinstance(raw, dict):
            raise ConfigError(f"config must be a JSON object, got {type(raw).__name__}")
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json needs a non-empty list 'layers' for Kamosun")
        cfg = cls(vocab=_get(raw, "vocab", int, "config.json"), width=_get(raw, "width", int, "config.json"),
                  norm_eps=_get(raw.get("norm"), "eps", float, "norm"),
                  residual_mult=_get(raw, "residual_mult", float, "config.json"),
                  layers=tuple(KamosunLayer.from_dict(l, f"layers[{i}]") for i, l in enumerate(layers)))
        cfg.validate()
        return cfg

    def validate(self) -> None:
        _positive(self, ("vocab", "width", "norm_eps"), "config.json")
        if not self.layers:
            raise ConfigError("a Kamosun model needs at least one layer")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}].mixer"
            layer.mixer.validate(where)
            if layer.mlp is not None:
                layer.mlp.validate(f"layers[{i}].mlp")
            src = getattr(layer.mixer, "kv_from", None)
            if src is None:
                continue
            if not 0 <= src < i or self.layers[src].type != "attention" or self.layers[src].mixer.kv_from is not None:
                raise ConfigError(f"{where}.kv_from {src} must name an earlier attention layer with keys and "
                                  "values of its own")
            mine, theirs = layer.mixer, self.layers[src].mixer
            if (mine.kv_heads, mine.dim, mine.vdim) != (theirs.kv_heads, theirs.dim, theirs.vdim):
                raise ConfigError(f"{where}: kv_heads, dim and vdim must equal those of layer {src}, whose keys "
                                  "and values it reads")

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "layers": [l.to_dict() for l in self.layers],
                "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult, "vocab": self.vocab,
                "width": self.width}
