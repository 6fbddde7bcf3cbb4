"""Configuration of the Domelix architecture: a decoder whose layers read the residual stream once for both sub-layers
(mixer and feed-forward side by side, each behind a norm of its own), whose layers are listed one by one (softmax
attention with a distance bias and a sink beside lightning attention; the gated delta rule; retention), each with a
feed-forward of routed experts chosen within groups, or none.

config.json names the model with ``"architecture": "Domelix"`` and carries::

    vocab, width                 sizes of the embedding and of the residual stream
    norm: {eps}                  epsilon of every RMS norm
    layers: [ {type, mixer: {...}, mlp: {...} | null} ]

``type`` "parallel": left: {heads, kv_heads, dim, vdim, scale, bias_max}, right: {heads, dim, vdim, decay: [per head]}.
``type`` "delta": heads, kv_heads, dim, vdim, conv (taps of the short convolutions).
``type`` "retention": heads, dim, vdim, decay: [per head], rot: {base, dims}.
``mlp``: {kind: "moe", expert: {ff}, router: {experts, top, groups: {count, keep}}}.
Every number comes from the file (the rows of a distance bias's table from its tensor); nothing is assumed about the
order or the count of the layers.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping, Optional, Tuple, Union

from .binupel_config import _int, _number
from .model_config import ConfigError, ModelConfig
from .zasalix_config import _object, _rotation

ARCHITECTURE = "Domelix"


@dataclass(frozen=True)
class BiasedAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    bias_max: float


@dataclass(frozen=True)
class DecayedMemory:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]


@dataclass(frozen=True)
class Retention(DecayedMemory):
    rot_base: float = 0.0
    rot_dims: int = 0


@dataclass(frozen=True)
class ParallelMixer:
    left: BiasedAttention
    right: DecayedMemory


@dataclass(frozen=True)
class GatedDelta:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass(frozen=True)
class GroupedExperts:
    experts: int
    top: int
    groups: int
    keep: int
    expert_ff: int


@dataclass(frozen=True)
class DomelixLayer:
    type: str
    mixer: Union[ParallelMixer, GatedDelta, Retention]
    mlp: Optional[GroupedExperts]


def _grouped_heads(where: str, m: Mapping[str, Any]) -> Tuple[int, int]:
    heads, kv_heads = _int(where, m, "heads"), _int(where, m, "kv_heads")
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}: {heads} heads are not a multiple of {kv_heads} kv_heads")
    return heads, kv_heads


def _attention(where: str, m: Mapping[str, Any]) -> BiasedAttention:
    heads, kv_heads = _grouped_heads(where, m)
    most = _number(where, m, "bias_max")
    if most <= 0:
        raise ConfigError(f"config.json: {where}: bias_max must be positive, got {most!r}")
    return BiasedAttention(heads, kv_heads, _int(where, m, "dim"), _int(where, m, "vdim"), _number(where, m, "scale"), most)


def _decay(where: str, m: Mapping[str, Any], heads: int) -> Tuple[float, ...]:
    values = m.get("decay")
    if (not isinstance(values, (list, tuple)) or len(values) != heads
            or any(isinstance(v, bool) or not isinstance(v, (int, float)) or not 0.0 <= v <= 1.0 for v in values)):
        raise ConfigError(f"config.json: {where}: 'decay' must list one number between 0 and 1 for each of the {heads} heads")
    return tuple(float(v) for v in values)


def _memory(where: str, m: Mapping[str, Any]) -> DecayedMemory:
    heads = _int(where, m, "heads")
    return DecayedMemory(heads, _int(where, m, "dim"), _int(where, m, "vdim"), _decay(where, m, heads))


def _retention(where: str, m: Mapping[str, Any]) -> Retention:
    heads, dim = _int(where, m, "heads"), _int(where, m, "dim")
    base, dims = _rotation(where, m, dim)
    return Retention(heads, dim, _int(where, m, "vdim"), _decay(where, m, heads), base, dims)


def _delta(where: str, m: Mapping[str, Any]) -> GatedDelta:
    heads, kv_heads = _grouped_heads(where, m)
    return GatedDelta(heads, kv_heads, _int(where, m, "dim"), _int(where, m, "vdim"), _int(where, m, "conv"))


def _mlp(where: str, mlp: Any) -> Optional[GroupedExperts]:
    if mlp is None:
        return None
    if not isinstance(mlp, Mapping) or mlp.get("kind") != "moe":
        raise ConfigError(f"config.json: {where}: mlp must be null or of kind 'moe', got {mlp!r}")
    router = _object(where, mlp, "router")
    at = f"{where}.router"
    experts, top = _int(at, router, "experts"), _int(at, router, "top")
    groups = _object(at, router, "groups")
    count, keep = _int(f"{at}.groups", groups, "count"), _int(f"{at}.groups", groups, "keep")
    if experts % count or keep > count:
        raise ConfigError(f"config.json: {at}: {experts} experts in {count} groups of which {keep} are kept")
    if top > keep * (experts // count):
        raise ConfigError(f"config.json: {at}: top {top} exceeds the {keep * (experts // count)} experts of the kept groups")
    return GroupedExperts(experts, top, count, keep, _int(f"{where}.expert", _object(where, mlp, "expert"), "ff"))


MIXERS = ("parallel", "delta", "retention")


@dataclass(frozen=True)
class DomelixConfig(ModelConfig):
    vocab: int = 0
    width: int = 0
    norm_eps: float = 0.0
    layers: Tuple[DomelixLayer, ...] = field(default_factory=tuple)
    eos_token_id: Optional[int] = None

    @classmethod
    def from_dict(cls, data: Mapping[str, Any]) -> "DomelixConfig":
        vocab, width = _int("model", data, "vocab"), _int("model", data, "width")
        eps = _number("norm", _object("model", data, "norm"), "eps")
        if eps <= 0:
            raise ConfigError(f"config.json: norm.eps must be positive, got {eps!r}")
        entries = data.get("layers")
        if not isinstance(entries, (list, tuple)) or not entries:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, entry in enumerate(entries):
            where = f"layers[{i}]"
            if not isinstance(entry, Mapping) or not isinstance(entry.get("mixer"), Mapping):
                raise ConfigError(f"config.json: {where} must be an object with 'type' and 'mixer'")
            kind, m = entry.get("type"), entry["mixer"]
            if kind == "parallel":
                mixer = ParallelMixer(_attention(f"{where}.mixer.left", _object(f"{where}.mixer", m, "left")),
                                      _memory(f"{where}.mixer.right", _object(f"{where}.mixer", m, "right")))
            elif kind == "delta":
                mixer = _delta(f"{where}.mixer", m)
            elif kind == "retention":
                mixer = _retention(f"{where}.mixer", m)
            else:
                raise ConfigError(f"config.json: {where}: mixer type {kind!r} is not built (built: {', '.join(MIXERS)})")
            layers.append(DomelixLayer(kind, mixer, _mlp(f"{where}.mlp", entry.get("mlp"))))
        eos = data.get("eos_token_id")
        return cls(architecture=ARCHITECTURE, vocab=vocab, width=width, norm_eps=eps, layers=tuple(layers),
                   eos_token_id=eos if isinstance(eos, int) else None)

    def to_dict(self) -> dict:
        entries = []
        for layer in self.layers:
            a = layer.mixer
            if layer.type == "parallel":
                mixer = {"left": {"heads": a.left.heads, "kv_heads": a.left.kv_heads, "dim": a.left.dim, "vdim": a.left.vdim,
                                  "scale": a.left.scale, "bias_max": a.left.bias_max},
                         "right": {"heads": a.right.heads, "dim": a.right.dim, "vdim": a.right.vdim,
                                   "decay": list(a.right.decay)}}
            elif layer.type == "delta":
                mixer = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "conv": a.conv}
            else:
                mixer = {"heads": a.heads, "dim": a.dim, "vdim": a.vdim, "decay": list(a.decay),
                         "rot": {"base": a.rot_base, "dims": a.rot_dims}}
            e, mlp = layer.mlp, None
            if e is not None:
                mlp = {"kind": "moe", "expert": {"ff": e.expert_ff},
                       "router": {"experts": e.experts, "top": e.top, "groups": {"count": e.groups, "keep": e.keep}}}
            entries.append({"type": layer.type, "mixer": mixer, "mlp": mlp})
        d = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "layers": entries}
        if self.eos_token_id is not None:
            d["eos_token_id"] = self.eos_token_id
        return d
