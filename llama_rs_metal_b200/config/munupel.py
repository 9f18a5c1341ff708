"""Configuration of the Munupel decoder, read from its own config.json keys.

    {"architecture": "Munupel", "vocab": V, "width": W, "norm": {"eps": e},
     "layers": [{"type": "attention" | "attention_2", "mixer": {...}, "mlp": {"kind": "dense", "ff": F} | null,
                 "weights_of": j}, ...]}

Both mixers: heads, kv_heads, dim, vdim, scale, rot {dims, base, scaling {factor, original, fast, slow}}. An attention
mixer besides: softcap (a cap on its scores) and mask {size} (the chunk of positions a query sees); an
attention_2 mixer: mask {size, keep_first} (the window, and the first keys every query sees besides). Absent
rot, rot.scaling, softcap, mask, mask.keep_first and mlp switch that off. A layer with `weights_of` runs layer j's
tensors on a cache entry of its own and lists layer j's sizes. Every size and every constant that can differ
between models comes from here.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from ..errors import InvalidError, UnsupportedError
from .base import read_int
from .kikalix import _positive, _real, _table


@dataclass(frozen=True)
class ScaledRotation:
    dims: int
    base: float
    scaling: Optional[Tuple[float, float, float, float]] = None  # factor, original, fast, slow

    @classmethod
    def read(cls, m: Mapping[str, Any], where: str, dim: int) -> Optional["ScaledRotation"]:
        rot = m.get("rot")
        if not isinstance(rot, Mapping) or not read_int(rot, "dims", 0):
            return None
        where += "rot."
        dims, base = _positive(rot, "dims", where), _real(rot, "base", where)
        if dims % 2 or dims > dim or base <= 0:
            raise InvalidError(f"config.{where[:-1]}: dims must be even and at most dim, base positive")
        scaling = rot.get("scaling")
        if isinstance(scaling, Mapping):
            scaling = tuple(_real(scaling, key, where + "scaling.") for key in ("factor", "original", "fast", "slow"))
            if min(scaling) <= 0 or base == 1.0:
                raise InvalidError(f"config.{where}scaling: every number must be positive, and base not 1")
        else:
            scaling = None
        return cls(dims, base, scaling)

    def to_dict(self) -> dict:
        out = {"dims": self.dims, "base": self.base}
        if self.scaling is not None:
            out["scaling"] = dict(zip(("factor", "original", "fast", "slow"), self.scaling))
        return out


@dataclass(frozen=True)
class GatedAttentionConfig:
    """Both mixers: `softcap` belongs to attention, `keep_first` to attention_2; `span` is the chunk's size
    for attention, the window's for attention_2 (None: every earlier key is seen)."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[ScaledRotation]
    span: Optional[int]
    softcap: Optional[float] = None
    keep_first: int = 0

    @classmethod
    def read(cls, m: Mapping[str, Any], where: str, kind: str) -> "GatedAttentionConfig":
        heads, kv_heads, dim, vdim = (_positive(m, k, where) for k in ("heads", "kv_heads", "dim", "vdim"))
        if heads % kv_heads:
            raise InvalidError(f"config.{where}heads must be a multiple of kv_heads")
        mask = m.get("mask") if isinstance(m.get("mask"), Mapping) else None
        span = _positive(mask, "size", where + "mask.") if mask is not None else None
        softcap, keep_first = None, 0
        if kind == "attention" and m.get("softcap") is not None:
            softcap = _real(m, "softcap", where)
            if softcap <= 0:
                raise InvalidError(f"config.{where}softcap must be positive")
        if kind == "attention_2" and mask is not None:
            keep_first = read_int(mask, "keep_first", 0)
            if keep_first < 0:
                raise InvalidError(f"config.{where}mask.keep_first cannot be negative")
        return cls(heads, kv_heads, dim, vdim, _real(m, "scale", where), ScaledRotation.read(m, where, dim), span,
                   softcap, keep_first)

    def to_dict(self) -> dict:
        out = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.rot is not None:
            out["rot"] = self.rot.to_dict()
        if self.span is not None:
            out["mask"] = {"size": self.span, **({"keep_first": self.keep_first} if self.keep_first else {})}
        if self.softcap is not None:
            out["softcap"] = self.softcap
        return out


KINDS = ("attention", "attention_2")


@dataclass(frozen=True)
class MunupelLayer:
    kind: str  # one of KINDS
    mixer: GatedAttentionConfig
    ff: Optional[int]
    weights_of: Optional[int] = None

    def to_dict(self) -> dict:
        out = {"type": self.kind, "mixer": self.mixer.to_dict(),
               "mlp": {"kind": "dense", "ff": self.ff} if self.ff is not None else None}
        if self.weights_of is not None:
            out["weights_of"] = self.weights_of
        return out


@dataclass(frozen=True)
class MunupelConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[MunupelLayer, ...]
    architecture: str = "Munupel"

    @classmethod
    def from_dict(cls, root: Mapping[str, Any]) -> "MunupelConfig":
        vocab, width = _positive(root, "vocab", ""), _positive(root, "width", "")
        eps = _real(_table(root, "norm", ""), "eps", "norm.")
        if eps <= 0:
            raise InvalidError("config.norm.eps must be positive")
        listed = root.get("layers")
        if not isinstance(listed, list) or not listed or len(listed) > 1024:
            raise InvalidError("config.layers must list 1 to 1024 layers")
        layers = []
        for i, item in enumerate(listed):
            where = f"layers[{i}]."
            if not isinstance(item, Mapping):
                raise InvalidError(f"config.layers[{i}] must be an object")
            kind = item.get("type")
            if kind not in KINDS:
                raise UnsupportedError(f"config.{where}type {kind!r}: built are {', '.join(KINDS)}")
            mixer = GatedAttentionConfig.read(_table(item, "mixer", where), where + "mixer.", kind)
            mlp, ff = item.get("mlp"), None
            if mlp is not None:
                if not isinstance(mlp, Mapping):
                    raise InvalidError(f"config.{where}mlp must be an object or null")
                if mlp.get("kind") != "dense":
                    raise UnsupportedError(f"config.{where}mlp.kind {mlp.get('kind')!r}: only \"dense\" is built")
                ff = _positive(mlp, "ff", where + "mlp.")
            other = read_int(item, "weights_of", None) if item.get("weights_of") is not None else None
            layers.append(MunupelLayer(kind, mixer, ff, other))
        config = cls(vocab, width, eps, tuple(layers))
        for i, layer in enumerate(layers):
            owner = layers[config.owner(i)]
            if (owner.kind, owner.mixer, owner.ff) != (layer.kind, layer.mixer, layer.ff):
                raise InvalidError(f"config.layers[{i}].weights_of: the layers' sizes differ")
        return config

    def owner(self, i: int) -> int:
        """The layer whose tensors layer i runs."""
        at, steps = i, 0
        while self.layers[at].weights_of is not None:
            at, steps = self.layers[at].weights_of, steps + 1
            if not 0 <= at < len(self.layers) or steps > len(self.layers):
                raise InvalidError(f"config.layers[{i}].weights_of must lead to a layer with tensors of its own")
        return at

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                "layers": [layer.to_dict() for layer in self.layers]}
