"""Configuration of the Gesuvik decoder (``"architecture": "Gesuvik"``).

A Gesuvik ``config.json`` is nested: ``vocab``, ``width``, ``norm.eps``, ``logit_scale``, ``logit_softcap`` and a list
``layers`` whose entries name their mixer (``type``: ``attention``, ``latent_attention`` or ``retention``), the mixer's
sizes and constants (``mixer``) and the routed experts behind it (``mlp``, or null for a layer without them).  An entry
with ``weights_of`` has no tensors of its own: it runs another layer once more, with a cache or state of its own.
Every size and every constant that can differ between two models of the design is read from the file; nothing is
filled in that the file does not give.
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
            raise ConfigError(f"config.json lacks the required key {where}.{name} for Gesuvik")
        return default
    return _coerce(f"{where}.{name}", raw[name], kind)


def _positive(obj, names, where):
    for name in names:
        if not getattr(obj, name) > 0:
            raise ConfigError(f"{where}.{name} must be positive, got {getattr(obj, name)}")


def _window(raw, where) -> Optional[int]:
    """``mask.size``: a token sees itself and the size - 1 tokens before it (no mask: every earlier token)."""
    mask = raw.get("mask")
    return None if mask is None else _get(mask, "size", int, where + ".mask")


@dataclasses.dataclass(frozen=True)
class RotationScaling:
    """``rot.scaling`` (YaRN): slow pairs turn ``factor`` times slower."""
    factor: float
    original: float
    fast: float
    slow: float

    @classmethod
    def from_dict(cls, raw, where):
        g = lambda n: _get(raw, n, float, where)
        return cls(factor=g("factor"), original=g("original"), fast=g("fast"), slow=g("slow"))

    def to_dict(self):
        return dataclasses.asdict(self)


@dataclasses.dataclass(frozen=True)
class Rotation:
    """``rot`` of a mixer."""
    dims: int
    base: float
    scaling: Optional[RotationScaling] = None

    @classmethod
    def from_dict(cls, raw, where):
        if raw is None:
            return None
        scaling = raw.get("scaling") if isinstance(raw, dict) else None
        return cls(dims=_get(raw, "dims", int, where), base=_get(raw, "base", float, where),
                   scaling=None if scaling is None else RotationScaling.from_dict(scaling, where + ".scaling"))

    def to_dict(self):
        out = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            out["scaling"] = self.scaling.to_dict()
        return out

    def validate(self, where, most):
        if self.dims < 0 or self.dims % 2 or self.dims > most:
            raise ConfigError(f"{where}.dims {self.dims} must be even and at most {most}")
        if not self.base > 0 or (self.scaling is not None and self.base == 1):
            raise ConfigError(f"{where}.base must be positive (and not 1 under a scaling)")
        if self.scaling is not None:
            _positive(self.scaling, ("factor", "original", "fast", "slow"), where + ".scaling")


@dataclasses.dataclass(frozen=True)
class GesuvikAttention:
    """``layers[i].mixer`` of an ``attention`` layer."""
    heads: int
    kv_heads: int
    dim: int                     # query / key size per head
    vdim: int                    # value size per head
    scale: float
    window: Optional[int]
    rot: Optional[Rotation]

    @classmethod
    def from_dict(cls, raw, where):
        g = lambda n, k=int: _get(raw, n, k, where)
        return cls(heads=g("heads"), kv_heads=g("kv_heads"), dim=g("dim"), vdim=g("vdim"), scale=g("scale", float),
                   window=_window(raw, where), rot=Rotation.from_dict(raw.get("rot"), where + ".rot"))

    def to_dict(self):
        out = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale, "vdim": self.vdim}
        return _with_mask_and_rot(out, self)

    def validate(self, where):
        _positive(self, ("heads", "kv_heads", "dim", "vdim"), where)
        if self.heads % self.kv_heads:
            raise ConfigError(f"{where}: heads {self.heads} is not a multiple of kv_heads {self.kv_heads}")
        _check_mask_and_rot(self, where, self.dim)


@dataclasses.dataclass(frozen=True)
class GesuvikLatentAttention:
    """``layers[i].mixer`` of a ``latent_attention`` layer."""
    heads: int
    dim: int                     # unrotated query / key size per head
    rot_dim: int                 # rotated query / key size
    vdim: int                    # value size per head
    kv_rank: int
    scale: float
    window: Optional[int]
    rot: Optional[Rotation]

    @classmethod
    def from_dict(cls, raw, where):
        g = lambda n, k=int: _get(raw, n, k, where)
        return cls(heads=g("heads"), dim=g("dim"), rot_dim=g("rot_dim"), vdim=g("vdim"), kv_rank=g("kv_rank"),
                   scale=g("scale", float), window=_window(raw, where),
                   rot=Rotation.from_dict(raw.get("rot"), where + ".rot"))

    def to_dict(self):
        out = {"dim": self.dim, "heads": self.heads, "kv_rank": self.kv_rank, "rot_dim": self.rot_dim,
               "scale": self.scale, "vdim": self.vdim}
        return _with_mask_and_rot(out, self)

    def validate(self, where):
        _positive(self, ("heads", "dim", "vdim", "kv_rank"), where)
        if self.rot_dim < 0:
            raise ConfigError(f"{where}.rot_dim must not be negative")
        _check_mask_and_rot(self, where, self.rot_dim)


def _with_mask_and_rot(out, m):
    if m.window is not None:
        out["mask"] = {"size": m.window}
    if m.rot is not None:
        out["rot"] = m.rot.to_dict()
    return out


def _check_mask_and_rot(m, where, most):
    if m.window is not None and m.window < 1:
        raise ConfigError(f"{where}: mask.size must be at least 1")
    if m.rot is not None:
        m.rot.validate(where + ".rot", most)


@dataclasses.dataclass(frozen=True)
class GesuvikRetention:
    """``layers[i].mixer`` of a ``retention`` layer."""
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    rot: Optional[Rotation]

    @classmethod
    def from_dict(cls, raw, where):
        g = lambda n: _get(raw, n, int, where)
        decay = raw.get("decay") if isinstance(raw, dict) else None
        if not isinstance(decay, list):
            raise ConfigError(f"config.json needs {where}.decay: a list with one number per head")
        return cls(heads=g("heads"), dim=g("dim"), vdim=g("vdim"),
                   decay=tuple(_coerce(f"{where}.decay", x, "float") for x in decay),
                   rot=Rotation.from_dict(raw.get("rot"), where + ".rot"))

    def to_dict(self):
        out = {"decay": list(self.decay), "dim": self.dim, "heads": self.heads, "vdim": self.vdim}
        if self.rot is not None:
            out["rot"] = self.rot.to_dict()
        return out

    def validate(self, where):
        _positive(self, ("heads", "dim", "vdim"), where)
        if len(self.decay) != self.heads:
            raise ConfigError(f"{where}.decay holds {len(self.decay)} numbers for {self.heads} heads")
        if self.rot is not None:
            self.rot.validate(where + ".rot", self.dim)


@dataclasses.dataclass(frozen=True)
class ClampedExpert:
    """One expert, or the shared expert: a gated feed-forward whose halves are clamped."""
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
class GesuvikExperts:
    """``layers[i].mlp``: routed experts, ``identity`` of them without tensors."""
    experts: int
    identity: int
    top: int
    expert: ClampedExpert
    shared: Optional[ClampedExpert]

    @classmethod
    def from_dict(cls, raw, where):
        kind = _get(raw, "kind", str, where)
        if kind != "moe":
            raise ConfigError(f"{where}.kind is {kind!r}; Gesuvik has the feed-forward moe")
        g = lambda n, d=dataclasses.MISSING: _get(raw.get("router"), n, int, where + ".router", d)
        shared = raw.get("shared")
        return cls(experts=g("experts"), identity=g("identity", 0), top=g("top"),
                   expert=ClampedExpert.from_dict(raw.get("expert"), where + ".expert"),
                   shared=None if shared is None else ClampedExpert.from_dict(shared, where + ".shared"))

    def to_dict(self):
        out = {"expert": self.expert.to_dict(), "kind": "moe",
               "router": {"experts": self.experts, "identity": self.identity, "top": self.top}}
        if self.shared is not None:
            out["shared"] = self.shared.to_dict()
        return out

    def validate(self, where):
        _positive(self, ("experts", "top"), where + ".router")
        if self.identity < 0:
            raise ConfigError(f"{where}.router.identity must not be negative")
        if self.top > self.experts + self.identity:
            raise ConfigError(f"{where}.router: top {self.top} exceeds the {self.experts} experts and {self.identity} "
                              "identity experts")
        self.expert.validate(where + ".expert")
        if self.shared is not None:
            self.shared.validate(where + ".shared")


MIXER_TYPES = {"attention": GesuvikAttention, "latent_attention": GesuvikLatentAttention, "retention": GesuvikRetention}
GesuvikMixer = Union[GesuvikAttention, GesuvikLatentAttention, GesuvikRetention]


@dataclasses.dataclass(frozen=True)
class GesuvikLayer:
    type: str
    mixer: GesuvikMixer
    mlp: Optional[GesuvikExperts]
    weights_of: Optional[int] = None

    @classmethod
    def from_dict(cls, raw, where):
        kind = _get(raw, "type", str, where)
        if kind not in MIXER_TYPES:
            raise ConfigError(f"{where}.type is {kind!r}; Gesuvik has the mixers {', '.join(sorted(MIXER_TYPES))}")
        if not isinstance(raw.get("mixer"), dict):
            raise ConfigError(f"config.json lacks the required record {where}.mixer for Gesuvik")
        mlp = raw.get("mlp")
        return cls(type=kind, mixer=MIXER_TYPES[kind].from_dict(raw["mixer"], where + ".mixer"),
                   mlp=None if mlp is None else GesuvikExperts.from_dict(mlp, where + ".mlp"),
                   weights_of=_get(raw, "weights_of", int, where, None))

    def to_dict(self):
        out = {"mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict(), "type": self.type}
        if self.weights_of is not None:
            out["weights_of"] = self.weights_of
        return out


@dataclasses.dataclass(frozen=True)
class GesuvikConfig(ModelConfig):
    architecture = "Gesuvik"

    vocab: int = 0
    width: int = 0
    norm_eps: float = 0.0
    logit_scale: float = 1.0
    logit_softcap: float = 0.0
    layers: Tuple[GesuvikLayer, ...] = ()

    @classmethod
    def from_dict(cls, raw: dict) -> "GesuvikConfig":
        if not isinstance(raw, dict):
            raise ConfigError(f"config must be a JSON object, got {type(raw).__name__}")
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json needs a non-empty list 'layers' for Gesuvik")
        g = lambda n, k: _get(raw, n, k, "config.json")
        cfg = cls(vocab=g("vocab", int), width=g("width", int), norm_eps=_get(raw.get("norm"), "eps", float, "norm"),
                  logit_scale=g("logit_scale", float), logit_softcap=g("logit_softcap", float),
                  layers=tuple(GesuvikLayer.from_dict(l, f"layers[{i}]") for i, l in enumerate(layers)))
        cfg.validate()
        return cfg

    def owner(self, i: int) -> int:
        """The layer whose tensors layer ``i`` uses."""
        while self.layers[i].weights_of is not None:
            i = self.layers[i].weights_of
        return i

    def validate(self) -> None:
        _positive(self, ("vocab", "width", "norm_eps", "logit_softcap"), "config.json")
        if not self.layers:
            raise ConfigError("a Gesuvik model needs at least one layer")
        for i, layer in enumerate(self.layers):
            src = layer.weights_of
            if src is not None:
                chain = {i}
                while src is not None:           # (a layer that borrows may name one that borrows too)
                    if not 0 <= src < len(self.layers) or src in chain:
                        raise ConfigError(f"layers[{i}].weights_of must lead to another layer with tensors of its own")
                    chain.add(src)
                    src = self.layers[src].weights_of
                src = layer.weights_of
                theirs = self.layers[src]
                if (layer.type, layer.mixer, layer.mlp) != (theirs.type, theirs.mixer, theirs.mlp):
                    raise ConfigError(f"layers[{i}]: type, mixer and mlp must equal those of layer {src}, whose weights "
                                      "it uses")
            layer.mixer.validate(f"layers[{i}].mixer")
            if layer.mlp is not None:
                layer.mlp.validate(f"layers[{i}].mlp")

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "layers": [l.to_dict() for l in self.layers],
                "logit_scale": self.logit_scale, "logit_softcap": self.logit_softcap, "norm": {"eps": self.norm_eps},
                "vocab": self.vocab, "width": self.width}
