"""Typed configuration of the Fipadra architecture, read from config.json.

config.json names the architecture by an `architecture` string and lists the layers one by one: each entry gives its
`type` (which mixer: `retention`, `delta` or `latent_attention`), the mixer's sizes and constants (`mixer`) and its
feed-forward (`mlp`: a dense unit, a routed mixture of experts, or null for none).  `norm` gives the norms' epsilon,
`logit_scale` a factor on the logits.  Every size and every constant that can differ between two models of the design is
read from there; nothing is assumed equal between layers, and what config.json does not mention is not there (no window,
no rotation, no groups of experts, no identity experts, no shared unit).  A value of the wrong kind, a missing size and
an unknown mixer or feed-forward kind are refused by name; keys this reader does not know are kept in `ignored` and have
no effect.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Any, Dict, Optional, Tuple

from .base import ConfigError, ModelConfig, _is_int
from .buzetar import DeltaMixer, LatentMixer      # the same two mixers, with the same sizes

MIXER_TYPES = ("retention", "delta", "latent_attention")


def _int(d: Dict[str, Any], key: str, where: str, minimum: int = 1) -> int:
    v = d.get(key)
    if not _is_int(v) or v < minimum:
        raise ConfigError(f"fipadra: {where}.{key} must be an integer >= {minimum}, got {v!r}")
    return int(v)


def _real(d: Dict[str, Any], key: str, where: str) -> float:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, (int, float)) or not math.isfinite(float(v)):
        raise ConfigError(f"fipadra: {where}.{key} must be a finite number, got {v!r}")
    return float(v)


def _obj(d: Dict[str, Any], key: str, where: str) -> Dict[str, Any]:
    v = d.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"fipadra: {where}.{key} must be an object, got {v!r}")
    return v


def _rotation(m: Dict[str, Any], where: str, width: int, what: str) -> Tuple[float, int]:
    """(base, rotated width); a mixer without `rot` rotates nothing."""
    if m.get("rot") is None:
        return 10000.0, 0
    rot = _obj(m, "rot", where)
    dims = _int(rot, "dims", where + ".rot", minimum=0)
    if dims % 2 or dims > width:
        raise ConfigError(f"fipadra: {where}.rot.dims must be even and at most {what} ({width}), got {dims}")
    base = _real(rot, "base", where + ".rot")
    if not base > 0:
        raise ConfigError(f"fipadra: {where}.rot.base must be positive, got {base!r}")
    return base, dims


@dataclass(frozen=True)
class RetentionMixer:
    """Linear attention with a constant decay per head; q and k rotated in the two-halves pairing."""
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    rot_base: float = 10000.0
    rot_dims: int = 0

    def to_dict(self) -> Dict[str, Any]:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay),
                "rot": {"base": self.rot_base, "dims": self.rot_dims}}


@dataclass(frozen=True)
class DenseMlp:
    ff: int

    def to_dict(self) -> Dict[str, Any]:
        return {"kind": "dense", "ff": self.ff}


@dataclass(frozen=True)
class ClampedUnit:
    """A clamped gated unit (an expert, or the shared unit): its inner width and its limit."""
    ff: int
    limit: float

    def to_dict(self) -> Dict[str, Any]:
        return {"ff": self.ff, "limit": self.limit}


@dataclass(frozen=True)
class RoutedMlp:
    """`experts` clamped units and `identity` experts that give their input back, `top` of them a token.  The router's
    outputs (experts, then identity experts) form `group_count` equal groups of neighbours of which a token keeps
    `group_keep`; the chosen weights sum to `scale`.  A shared unit under a sigmoid gate beside them, or none."""
    experts: int
    top: int
    expert: ClampedUnit
    identity: int = 0
    group_count: int = 1
    group_keep: int = 1
    scale: float = 1.0
    shared: Optional[ClampedUnit] = None

    @property
    def outputs(self) -> int:
        return self.experts + self.identity

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"kind": "moe", "expert": self.expert.to_dict(),
                             "router": {"experts": self.experts, "identity": self.identity, "top": self.top, "scale": self.scale,
                                        "groups": {"count": self.group_count, "keep": self.group_keep}}}
        if self.shared is not None:
            d["shared"] = self.shared.to_dict()
        return d


@dataclass(frozen=True)
class FipadraLayer:
    type: str
    mixer: Any                     # RetentionMixer, DeltaMixer or LatentMixer
    mlp: Any                       # DenseMlp, RoutedMlp or None

    def to_dict(self) -> Dict[str, Any]:
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}


def _read_mixer(kind: Any, m: Dict[str, Any], where: str):
    if kind == "retention":
        heads, dim = _int(m, "heads", where), _int(m, "dim", where)
        decay = m.get("decay")
        if not isinstance(decay, list) or len(decay) != heads or any(
                isinstance(x, bool) or not isinstance(x, (int, float)) or not math.isfinite(float(x)) for x in decay):
            raise ConfigError(f"fipadra: {where}.decay must be a list of {heads} numbers (one per head), got {decay!r}")
        base, dims = _rotation(m, where, dim, "dim")
        return RetentionMixer(heads, dim, _int(m, "vdim", where), tuple(float(x) for x in decay), base, dims)
    if kind == "delta":
        heads, kv_heads = _int(m, "heads", where), _int(m, "kv_heads", where)
        if heads % kv_heads:
            raise ConfigError(f"fipadra: {where}.heads ({heads}) must be a multiple of kv_heads ({kv_heads})")
        return DeltaMixer(heads, kv_heads, _int(m, "dim", where), _int(m, "vdim", where), _int(m, "conv", where))
    if kind == "latent_attention":
        rot_dim = _int(m, "rot_dim", where, minimum=0)
        base, dims = _rotation(m, where, rot_dim, "rot_dim")
        window = None if m.get("mask") is None else _int(_obj(m, "mask", where), "size", where + ".mask")
        return LatentMixer(_int(m, "heads", where), _int(m, "dim", where), rot_dim, _int(m, "vdim", where), _int(m, "q_rank", where),
                           _int(m, "kv_rank", where), _real(m, "scale", where), base, dims, window)
    raise ConfigError(f"fipadra: {where}: mixer type {kind!r} is not one of {list(MIXER_TYPES)}")


def _read_unit(raw: Dict[str, Any], key: str, where: str) -> ClampedUnit:
    d = _obj(raw, key, where)
    return ClampedUnit(_int(d, "ff", f"{where}.{key}"), _real(d, "limit", f"{where}.{key}"))


def _read_mlp(raw: Any, where: str):
    if raw is None:
        return None
    if not isinstance(raw, dict):
        raise ConfigError(f"fipadra: {where} must be an object or null")
    kind = raw.get("kind")
    if kind == "dense":
        return DenseMlp(_int(raw, "ff", where))
    if kind == "moe":
        rw = where + ".router"
        router = _obj(raw, "router", where)
        experts, top = _int(router, "experts", rw), _int(router, "top", rw)
        identity = _int(router, "identity", rw, minimum=0) if router.get("identity") is not None else 0
        count = keep = 1
        if router.get("groups") is not None:
            groups = _obj(router, "groups", rw)
            count, keep = _int(groups, "count", rw + ".groups"), _int(groups, "keep", rw + ".groups")
        outputs = experts + identity
        if outputs % count:
            raise ConfigError(f"fipadra: {rw}: {outputs} router outputs do not form {count} equal groups")
        if keep > count:
            raise ConfigError(f"fipadra: {rw}.groups.keep ({keep}) exceeds the number of groups ({count})")
        if top > keep * (outputs // count):
            raise ConfigError(f"fipadra: {rw}.top ({top}) exceeds the experts that can be chosen ({keep * (outputs // count)})")
        scale = _real(router, "scale", rw) if router.get("scale") is not None else 1.0
        shared = None if raw.get("shared") is None else _read_unit(raw, "shared", where)
        return RoutedMlp(experts, top, _read_unit(raw, "expert", where), identity, count, keep, scale, shared)
    raise ConfigError(f"fipadra: {where}.kind {kind!r} is not supported (\"dense\", \"moe\")")


@dataclass(frozen=True)
class FipadraConfig(ModelConfig):
    vocab: int
    width: int
    layers: Tuple[FipadraLayer, ...]
    norm_eps: float
    logit_scale: float = 1.0
    ignored: Tuple[str, ...] = field(default=(), compare=False)

    model_type = "fipadra"
    class_name = "Fipadra"

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "FipadraConfig":
        if raw.get("architecture") != "Fipadra":
            raise ConfigError(f"fipadra: config.json names architecture {raw.get('architecture')!r}")
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError("fipadra: layers must be a list with at least one layer")
        layers = []
        for i, entry in enumerate(layers_raw):
            where = f"layers[{i}]"
            if not isinstance(entry, dict):
                raise ConfigError(f"fipadra: {where} must be an object")
            kind = entry.get("type")
            mixer = _read_mixer(kind, _obj(entry, "mixer", where), where + ".mixer")
            layers.append(FipadraLayer(kind, mixer, _read_mlp(entry.get("mlp"), where + ".mlp")))
        eps = _real(_obj(raw, "norm", "config"), "eps", "norm")
        if not eps >= 0:
            raise ConfigError("fipadra: norm.eps must not be negative")
        scale = _real(raw, "logit_scale", "config") if raw.get("logit_scale") is not None else 1.0
        known = {"architecture", "layers", "norm", "logit_scale", "vocab", "width", "torch_dtype"}
        return cls(vocab=_int(raw, "vocab", "config"), width=_int(raw, "width", "config"), layers=tuple(layers), norm_eps=eps,
                   logit_scale=scale, ignored=tuple(sorted(k for k in raw if k not in known)))

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": "Fipadra", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "logit_scale": self.logit_scale, "layers": [layer.to_dict() for layer in self.layers]}
