"""Configuration of the Zasitar architecture: a decoder with a norm on the sub-layers' outputs alone and a learned scale per
feature behind it, whose layers are listed one by one (RWKV-style time mixing, or windowed attention whose keys and values
may be another layer's), each with a dense feed-forward, routed experts beside a shared one, or none.

config.json names the model with ``"architecture": "Zasitar"`` and carries::

    vocab, width                 sizes of the embedding and of the residual stream
    norm: {eps}                  epsilon of every RMS norm
    layers: [ {type, mixer: {...}, mlp: {...} | null} ]

``type`` "wkv": heads, dim (the rank of the decay's projection is what the stored tensors say).
``type`` "attention": heads, kv_heads, dim, vdim, scale, mask: {size}, rot: {base, dims, scaling: {factor, low, high,
original} | absent}, and optionally kv_from: the number of an earlier attention layer with keys of its own (and the same
head counts, sizes and rotation), whose keys and values this layer reads.
``mlp``: {kind: "dense", ff} or {kind: "moe", expert: {ff, limit}, router: {experts, top}, shared: {ff, limit} | absent}.
Every number comes from the file; nothing is assumed about the order or the count of the layers.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping, Optional, Tuple, Union

from .binupel_config import _int, _number
from .domelix_config import _grouped_heads
from .model_config import ConfigError, ModelConfig
from .zasalix_config import DenseFF, _count, _object, _rotation

ARCHITECTURE = "Zasitar"


@dataclass(frozen=True)
class TimeMixing:
    heads: int
    dim: int


@dataclass(frozen=True)
class BandScaling:
    factor: float
    low: float
    high: float
    original: float


@dataclass(frozen=True)
class SharedKeyAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int
    rot_base: float
    rot_dims: int
    rot_scaling: Optional[BandScaling] = None
    kv_from: Optional[int] = None

    @property
    def kept(self):
        """What a layer and the one whose keys it reads have in common."""
        return (self.heads, self.kv_heads, self.dim, self.vdim, self.rot_base, self.rot_dims, self.rot_scaling)


@dataclass(frozen=True)
class LimitedFF:
    ff: int
    limit: float


@dataclass(frozen=True)
class LimitedExperts:
    experts: int
    top: int
    expert: LimitedFF
    shared: Optional[LimitedFF] = None


@dataclass(frozen=True)
class ZasitarLayer:
    type: str
    mixer: Union[TimeMixing, SharedKeyAttention]
    mlp: Union[DenseFF, LimitedExperts, None]


def _positive(where: str, data: Mapping[str, Any], key: str) -> float:
    value = _number(where, data, key)
    if value <= 0:
        raise ConfigError(f"config.json: {where}: '{key}' must be positive, got {value!r}")
    return value


def _scaling(where: str, rot: Mapping[str, Any]) -> Optional[BandScaling]:
    if rot.get("scaling") is None:
        return None
    s, at = _object(where, rot, "scaling"), f"{where}.scaling"
    out = BandScaling(_positive(at, s, "factor"), _number(at, s, "low"), _number(at, s, "high"), _positive(at, s, "original"))
    if out.high <= out.low:
        raise ConfigError(f"config.json: {at}: high {out.high!r} must exceed low {out.low!r}")
    return out


def _attention(where: str, m: Mapping[str, Any]) -> SharedKeyAttention:
    heads, kv_heads = _grouped_heads(where, m)
    dim = _int(where, m, "dim")
    base, dims = _rotation(where, m, dim)
    return SharedKeyAttention(heads, kv_heads, dim, _int(where, m, "vdim"), _number(where, m, "scale"),
                              _int(f"{where}.mask", _object(where, m, "mask"), "size"), base, dims,
                              _scaling(f"{where}.rot", m["rot"]),
                              None if m.get("kv_from") is None else _count(where, m, "kv_from"))


def _limited(where: str, data: Mapping[str, Any]) -> LimitedFF:
    return LimitedFF(_int(where, data, "ff"), _positive(where, data, "limit"))


def _mlp(where: str, mlp: Any) -> Union[DenseFF, LimitedExperts, None]:
    if mlp is None:
        return None
    if not isinstance(mlp, Mapping) or mlp.get("kind") not in ("dense", "moe"):
        raise ConfigError(f"config.json: {where}: mlp must be null or of kind 'dense' or 'moe', got {mlp!r}")
    if mlp["kind"] == "dense":
        return DenseFF(_int(where, mlp, "ff"))
    at, router = f"{where}.router", _object(where, mlp, "router")
    experts, top = _int(at, router, "experts"), _int(at, router, "top")
    if top > experts:
        raise ConfigError(f"config.json: {at}: top {top} of {experts} experts")
    shared = None if mlp.get("shared") is None else _limited(f"{where}.shared", _object(where, mlp, "shared"))
    return LimitedExperts(experts, top, _limited(f"{where}.expert", _object(where, mlp, "expert")), shared)


MIXERS = ("wkv", "attention")


@dataclass(frozen=True)
class ZasitarConfig(ModelConfig):
    vocab: int = 0
    width: int = 0
    norm_eps: float = 0.0
    layers: Tuple[ZasitarLayer, ...] = field(default_factory=tuple)
    eos_token_id: Optional[int] = None

    @classmethod
    def from_dict(cls, data: Mapping[str, Any]) -> "ZasitarConfig":
        vocab, width = _int("model", data, "vocab"), _int("model", data, "width")
        eps = _positive("norm", _object("model", data, "norm"), "eps")
        entries = data.get("layers")
        if not isinstance(entries, (list, tuple)) or not entries:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, entry in enumerate(entries):
            where = f"layers[{i}]"
            if not isinstance(entry, Mapping) or not isinstance(entry.get("mixer"), Mapping):
                raise ConfigError(f"config.json: {where} must be an object with 'type' and 'mixer'")
            kind, m = entry.get("type"), entry["mixer"]
            if kind == "wkv":
                mixer = TimeMixing(_int(f"{where}.mixer", m, "heads"), _int(f"{where}.mixer", m, "dim"))
            elif kind == "attention":
                mixer = _attention(f"{where}.mixer", m)
            else:
                raise ConfigError(f"config.json: {where}: mixer type {kind!r} is not built (built: {', '.join(MIXERS)})")
            if kind == "attention" and mixer.kv_from is not None:
                j = mixer.kv_from
                if not (j < i and layers[j].type == "attention" and layers[j].mixer.kv_from is None):
                    raise ConfigError(f"config.json: {where}: kv_from {j} must name an earlier attention layer with keys of its own")
                if layers[j].mixer.kept != mixer.kept:
                    raise ConfigError(f"config.json: {where}: kv_from {j}: heads, sizes and rotation must be layer {j}'s")
            layers.append(ZasitarLayer(kind, mixer, _mlp(f"{where}.mlp", entry.get("mlp"))))
        eos = data.get("eos_token_id")
        return cls(architecture=ARCHITECTURE, vocab=vocab, width=width, norm_eps=eps, layers=tuple(layers),
                   eos_token_id=eos if isinstance(eos, int) else None)

    def to_dict(self) -> dict:
        entries = []
        for layer in self.layers:
            a, e, mlp = layer.mixer, layer.mlp, None
            if layer.type == "wkv":
                mixer = {"heads": a.heads, "dim": a.dim}
            else:
                rot = {"base": a.rot_base, "dims": a.rot_dims}
                if a.rot_scaling is not None:
                    s = a.rot_scaling
                    rot["scaling"] = {"factor": s.factor, "low": s.low, "high": s.high, "original": s.original}
                mixer = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale,
                         "mask": {"size": a.window}, "rot": rot}
                if a.kv_from is not None:
                    mixer["kv_from"] = a.kv_from
            if isinstance(e, DenseFF):
                mlp = {"kind": "dense", "ff": e.ff}
            elif e is not None:
                mlp = {"kind": "moe", "expert": {"ff": e.expert.ff, "limit": e.expert.limit},
                       "router": {"experts": e.experts, "top": e.top}}
                if e.shared is not None:
                    mlp["shared"] = {"ff": e.shared.ff, "limit": e.shared.limit}
            entries.append({"type": layer.type, "mixer": mixer, "mlp": mlp})
        d = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "layers": entries}
        if self.eos_token_id is not None:
            d["eos_token_id"] = self.eos_token_id
        return d
