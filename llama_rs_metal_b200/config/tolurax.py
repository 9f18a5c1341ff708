"""Configuration of the Tolurax decoder, read from its own config.json keys.

    {"architecture": "Tolurax", "vocab": V, "width": W, "norm": {"eps": e}, "canon": {"taps": n},
     "logit_softcap": c, "loop": {"start": a, "stop": b, "times": m},
     "layers": [{"type": "delta" | "parallel", "mixer": {...}, "mlp": {"kind": "dense", "ff": F} | null}, ...]}

A delta mixer: heads, kv_heads, dim, vdim, conv (taps). A parallel mixer: left {heads, kv_heads, dim,
vdim, scale, rot {dims, base, scaling {factor, low, high, original}}, mask {size}}, right {heads, dim},
left_scale, right_scale. The inner rank of the right mixer's decay is no configuration key and is read
off the checkpoint's tensors (the optional key right.decay_rank gives it to the random-weights mode,
which has no checkpoint to ask). Absent canon, logit_softcap, loop, rot, rot.scaling and mask switch
that off. Every size and every constant that can differ between models comes from here.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from ..errors import InvalidError, UnsupportedError
from .base import read_int
from .kikalix import _positive, _real, _table


@dataclass(frozen=True)
class DeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    @classmethod
    def read(cls, m: Mapping[str, Any], where: str) -> "DeltaConfig":
        heads, kv_heads, dim, vdim, conv = (_positive(m, k, where) for k in ("heads", "kv_heads", "dim", "vdim", "conv"))
        if heads % kv_heads:
            raise InvalidError(f"config.{where}heads must be a multiple of kv_heads")
        return cls(heads, kv_heads, dim, vdim, conv)

    def to_dict(self) -> dict:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "conv": self.conv}


@dataclass(frozen=True)
class RotationConfig:
    dims: int
    base: float
    scaling: Optional[Tuple[float, float, float, float]] = None   # (factor, low, high, original)

    @classmethod
    def read(cls, parent: Mapping[str, Any], dim: int, where: str) -> Optional["RotationConfig"]:
        rot = parent.get("rot")
        if not isinstance(rot, Mapping) or not read_int(rot, "dims", 0):
            return None
        dims, base = read_int(rot, "dims", 0), _real(rot, "base", where + "rot.")
        if dims % 2 or dims > dim or base <= 0:
            raise InvalidError(f"config.{where}rot: dims must be even and at most dim, base positive")
        scaling = None
        if isinstance(rot.get("scaling"), Mapping):
            scaling = tuple(_real(rot["scaling"], k, where + "rot.scaling.") for k in ("factor", "low", "high", "original"))
            if min(scaling) <= 0:
                raise InvalidError(f"config.{where}rot.scaling: factor, low, high and original must be positive")
        return cls(dims, base, scaling)

    def to_dict(self) -> dict:
        out = {"dims": self.dims, "base": self.base}
        if self.scaling is not None:
            out["scaling"] = dict(zip(("factor", "low", "high", "original"), self.scaling))
        return out


@dataclass(frozen=True)
class SigmoidAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[RotationConfig]
    window: Optional[int]

    @classmethod
    def read(cls, m: Mapping[str, Any], where: str) -> "SigmoidAttentionConfig":
        heads, kv_heads, dim, vdim = (_positive(m, k, where) for k in ("heads", "kv_heads", "dim", "vdim"))
        if heads % kv_heads:
            raise InvalidError(f"config.{where}heads must be a multiple of kv_heads")
        window = _positive(m["mask"], "size", where + "mask.") if isinstance(m.get("mask"), Mapping) else None
        return cls(heads, kv_heads, dim, vdim, _real(m, "scale", where), RotationConfig.read(m, dim, where), window)

    def to_dict(self) -> dict:
        out = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.rot is not None:
            out["rot"] = self.rot.to_dict()
        if self.window is not None:
            out["mask"] = {"size": self.window}
        return out


@dataclass(frozen=True)
class TimeMixConfig:
    heads: int
    dim: int
    decay_rank: Optional[int] = None

    @classmethod
    def read(cls, m: Mapping[str, Any], where: str) -> "TimeMixConfig":
        rank = read_int(m, "decay_rank", None)
        return cls(_positive(m, "heads", where), _positive(m, "dim", where), rank if rank else None)

    def to_dict(self) -> dict:
        out = {"heads": self.heads, "dim": self.dim}
        if self.decay_rank is not None:
            out["decay_rank"] = self.decay_rank
        return out


@dataclass(frozen=True)
class ParallelConfig:
    left: SigmoidAttentionConfig
    right: TimeMixConfig
    left_scale: float
    right_scale: float

    @classmethod
    def read(cls, m: Mapping[str, Any], where: str) -> "ParallelConfig":
        return cls(SigmoidAttentionConfig.read(_table(m, "left", where), where + "left."),
                   TimeMixConfig.read(_table(m, "right", where), where + "right."),
                   _real(m, "left_scale", where), _real(m, "right_scale", where))

    def to_dict(self) -> dict:
        return {"left": self.left.to_dict(), "left_scale": self.left_scale, "right": self.right.to_dict(),
                "right_scale": self.right_scale}


MIXERS = {"delta": DeltaConfig, "parallel": ParallelConfig}


@dataclass(frozen=True)
class ToluraxLayer:
    kind: str  # a key of MIXERS
    mixer: Any
    ff: Optional[int]  # inner width of the dense feed-forward; None: no feed-forward

    def to_dict(self) -> dict:
        return {"type": self.kind, "mixer": self.mixer.to_dict(),
                "mlp": {"kind": "dense", "ff": self.ff} if self.ff is not None else None}


@dataclass(frozen=True)
class ToluraxConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[ToluraxLayer, ...]
    canon_taps: int = 0                    # 0: no input convolution
    logit_softcap: Optional[float] = None
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 1
    architecture: str = "Tolurax"

    @classmethod
    def from_dict(cls, root: Mapping[str, Any]) -> "ToluraxConfig":
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
            if kind not in MIXERS:
                raise UnsupportedError(f"config.{where}type {kind!r}: built are {', '.join(sorted(MIXERS))}")
            mixer = MIXERS[kind].read(_table(item, "mixer", where), where + "mixer.")
            mlp, ff = item.get("mlp"), None
            if mlp is not None:
                if not isinstance(mlp, Mapping):
                    raise InvalidError(f"config.{where}mlp must be an object or null")
                if mlp.get("kind") != "dense":
                    raise UnsupportedError(f"config.{where}mlp.kind {mlp.get('kind')!r}: built is \"dense\"")
                ff = _positive(mlp, "ff", where + "mlp.")
            layers.append(ToluraxLayer(kind, mixer, ff))
        canon = root.get("canon")
        taps = _positive(canon, "taps", "canon.") if isinstance(canon, Mapping) else 0
        cap = None
        if root.get("logit_softcap") is not None:
            cap = _real(root, "logit_softcap", "")
            if cap <= 0:
                raise InvalidError("config.logit_softcap must be positive")
        start, stop, times = 0, 0, 1
        loop = root.get("loop")
        if isinstance(loop, Mapping):
            start, stop = read_int(loop, "start"), read_int(loop, "stop")
            times = _positive(loop, "times", "loop.")
            if not 0 <= start <= stop <= len(layers) or times > 1024:
                raise InvalidError("config.loop: 0 <= start <= stop <= number of layers, times at most 1024")
        return cls(vocab, width, eps, tuple(layers), taps, cap, start, stop, times)

    @property
    def loops(self) -> bool:
        return self.loop_stop > self.loop_start

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
               "layers": [layer.to_dict() for layer in self.layers]}
        if self.canon_taps:
            out["canon"] = {"taps": self.canon_taps}
        if self.logit_softcap is not None:
            out["logit_softcap"] = self.logit_softcap
        if self.loops:
            out["loop"] = {"start": self.loop_start, "stop": self.loop_stop, "times": self.loop_times}
        return out
