"""Typed configuration of the Dikusun architecture, read from config.json.

config.json names the architecture by an `architecture` string and lists the layers one by one: each entry gives its
`type` (which mixer: `latent_attention`, `attention` or `gla`), the mixer's sizes and constants (`mixer`), its feed-forward
(`mlp`: a dense clamped unit, or null for none) and, for a layer without tensors of its own, `weights_of`: the layer whose
weights it uses (the rest of its entry repeats that layer's).  `norm` gives the norms' epsilon, `embedding` a factor on the
embedding.  Every size and every constant that can differ between two models of the design is read from there (the inner
width of the decay's low-rank pair from its tensors); nothing is assumed equal between layers, and what config.json does not
mention is not there (no window, no rotation, no cap on the scores).  A value of the wrong kind, a missing size and an unknown
mixer or feed-forward kind are refused by name; keys this reader does not know are kept in `ignored` and have no effect.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Any, Dict, Optional, Tuple

from .base import ConfigError, ModelConfig, _is_int

MIXER_TYPES = ("latent_attention", "attention", "gla")


def _int(d: Dict[str, Any], key: str, where: str, minimum: int = 1) -> int:
    v = d.get(key)
    if not _is_int(v) or v < minimum:
        raise ConfigError(f"dikusun: {where}.{key} must be an integer >= {minimum}, got {v!r}")
    return int(v)


def _real(d: Dict[str, Any], key: str, where: str) -> float:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, (int, float)) or not math.isfinite(float(v)):
        raise ConfigError(f"dikusun: {where}.{key} must be a finite number, got {v!r}")
    return float(v)


def _positive(d: Dict[str, Any], key: str, where: str) -> float:
    v = _real(d, key, where)
    if not v > 0:
        raise ConfigError(f"dikusun: {where}.{key} must be positive, got {v!r}")
    return v


def _obj(d: Dict[str, Any], key: str, where: str) -> Dict[str, Any]:
    v = d.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"dikusun: {where}.{key} must be an object, got {v!r}")
    return v


@dataclass(frozen=True)
class LatentMixer:
    """Latent attention without positions: queries and keys/values through normed latents of their own."""
    heads: int
    dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float

    def to_dict(self) -> Dict[str, Any]:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "q_rank": self.q_rank, "kv_rank": self.kv_rank,
                "scale": self.scale}


@dataclass(frozen=True)
class DifferentialMixer:
    """Differential softmax attention: two maps a head over the same values, a window, a cap on the scores."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    softcap: Optional[float] = None
    window: Optional[int] = None
    rot_base: float = 10000.0
    rot_dims: int = 0

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale,
                             "diff": self.diff, "rot": {"base": self.rot_base, "dims": self.rot_dims}}
        if self.softcap is not None:
            d["softcap"] = self.softcap
        if self.window is not None:
            d["mask"] = {"size": self.window}
        return d


@dataclass(frozen=True)
class GlaMixer:
    """Gated linear attention: a decay per key channel, the tau-th root of a sigmoid."""
    heads: int
    dim: int
    vdim: int
    tau: float
    decay_rank: Optional[int] = None      # the inner width of the decay's low-rank pair: the tensors' shapes give it; named
    #                                       only in a configuration that weights are made from

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "tau": self.tau}
        if self.decay_rank is not None:
            d["decay_rank"] = self.decay_rank
        return d


@dataclass(frozen=True)
class ClampedMlp:
    """A clamped gated unit: its inner width and its limit."""
    ff: int
    limit: float

    def to_dict(self) -> Dict[str, Any]:
        return {"kind": "dense", "ff": self.ff, "limit": self.limit}


@dataclass(frozen=True)
class DikusunLayer:
    type: str
    mixer: Any                        # LatentMixer, DifferentialMixer or GlaMixer
    mlp: Optional[ClampedMlp]
    weights_of: Optional[int] = None  # the layer whose tensors this one uses

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}
        if self.weights_of is not None:
            d["weights_of"] = self.weights_of
        return d


def _read_mixer(kind: Any, m: Dict[str, Any], where: str):
    if kind == "latent_attention":
        return LatentMixer(_int(m, "heads", where), _int(m, "dim", where), _int(m, "vdim", where), _int(m, "q_rank", where),
                           _int(m, "kv_rank", where), _real(m, "scale", where))
    if kind == "attention":
        heads, kv_heads, dim = _int(m, "heads", where), _int(m, "kv_heads", where), _int(m, "dim", where)
        if heads % kv_heads:
            raise ConfigError(f"dikusun: {where}.heads ({heads}) must be a multiple of kv_heads ({kv_heads})")
        base, dims = 10000.0, 0
        if m.get("rot") is not None:
            rot = _obj(m, "rot", where)
            dims, base = _int(rot, "dims", where + ".rot", minimum=0), _positive(rot, "base", where + ".rot")
            if dims % 2 or dims > dim:
                raise ConfigError(f"dikusun: {where}.rot.dims must be even and at most dim ({dim}), got {dims}")
        cap = None if m.get("softcap") is None else _positive(m, "softcap", where)
        window = None if m.get("mask") is None else _int(_obj(m, "mask", where), "size", where + ".mask")
        return DifferentialMixer(heads, kv_heads, dim, _int(m, "vdim", where), _real(m, "scale", where), _real(m, "diff", where), cap,
                                 window, base, dims)
    if kind == "gla":
        return GlaMixer(_int(m, "heads", where), _int(m, "dim", where), _int(m, "vdim", where), _positive(m, "tau", where),
                        None if m.get("decay_rank") is None else _int(m, "decay_rank", where))
    raise ConfigError(f"dikusun: {where}: mixer type {kind!r} is not one of {list(MIXER_TYPES)}")


def _read_mlp(raw: Any, where: str) -> Optional[ClampedMlp]:
    if raw is None:
        return None
    if not isinstance(raw, dict):
        raise ConfigError(f"dikusun: {where} must be an object or null")
    if raw.get("kind") != "dense":
        raise ConfigError(f"dikusun: {where}.kind {raw.get('kind')!r} is not supported (\"dense\")")
    return ClampedMlp(_int(raw, "ff", where), _real(raw, "limit", where))


@dataclass(frozen=True)
class DikusunConfig(ModelConfig):
    vocab: int
    width: int
    layers: Tuple[DikusunLayer, ...]
    norm_eps: float
    embedding_scale: float = 1.0
    ignored: Tuple[str, ...] = field(default=(), compare=False)

    model_type = "dikusun"
    class_name = "Dikusun"

    def owner(self, i: int) -> int:
        """The layer whose tensors layer i uses (i itself, or the end of the `weights_of` it names)."""
        while self.layers[i].weights_of is not None:
            i = self.layers[i].weights_of
        return i

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "DikusunConfig":
        if raw.get("architecture") != "Dikusun":
            raise ConfigError(f"dikusun: config.json names architecture {raw.get('architecture')!r}")
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError("dikusun: layers must be a list with at least one layer")
        layers = []
        for i, entry in enumerate(layers_raw):
            where = f"layers[{i}]"
            if not isinstance(entry, dict):
                raise ConfigError(f"dikusun: {where} must be an object")
            kind = entry.get("type")
            mixer = _read_mixer(kind, _obj(entry, "mixer", where), where + ".mixer")
            source = None if entry.get("weights_of") is None else _int(entry, "weights_of", where, minimum=0)
            if source is not None and (source >= len(layers_raw) or source == i):
                raise ConfigError(f"dikusun: {where}.weights_of must name another layer, got {source}")
            layers.append(DikusunLayer(kind, mixer, _read_mlp(entry.get("mlp"), where + ".mlp"), source))
        for i, layer in enumerate(layers):
            seen, j = {i}, i
            while layers[j].weights_of is not None:
                j = layers[j].weights_of
                if j in seen:
                    raise ConfigError(f"dikusun: layers[{i}].weights_of leads back to itself")
                seen.add(j)
            if (layer.type, layer.mixer, layer.mlp) != (layers[j].type, layers[j].mixer, layers[j].mlp):
                raise ConfigError(f"dikusun: layers[{i}] uses the weights of layer {j} but its entry differs from that layer's")
        eps = _real(_obj(raw, "norm", "config"), "eps", "norm")
        if not eps >= 0:
            raise ConfigError("dikusun: norm.eps must not be negative")
        scale = 1.0
        if raw.get("embedding") is not None and _obj(raw, "embedding", "config").get("scale") is not None:
            scale = _real(raw["embedding"], "scale", "embedding")
        known = {"architecture", "layers", "norm", "embedding", "vocab", "width", "torch_dtype"}
        return cls(vocab=_int(raw, "vocab", "config"), width=_int(raw, "width", "config"), layers=tuple(layers), norm_eps=eps,
                   embedding_scale=scale, ignored=tuple(sorted(k for k in raw if k not in known)))

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": "Dikusun", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "embedding": {"scale": self.embedding_scale}, "layers": [layer.to_dict() for layer in self.layers]}
