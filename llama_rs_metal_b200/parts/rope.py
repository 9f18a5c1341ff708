"""Rotary position encoding (split-half or adjacent pairs) with linear, llama3 and yarn frequency scaling."""
from __future__ import annotations

import math
from typing import List, Optional, Tuple

import torch

from ..errors import InvalidError, UnsupportedError
from ..registry import register_position_encoding
from .base import PositionEncoding


_shared_frequencies = {}  # (device, frequencies) -> float32 and float64 tensors on that device

@register_position_encoding("rope")
class RotaryEmbedding(PositionEncoding):
    """angle(position, pair i) = position * scale * theta^(-2i/R) / factor[i]
    (crates/metal-backend/src/shaders/attention.metal:16-20). The per-pair
    inverse frequency is computed once on the host in double precision and
    rounded to float32; the kernel forms the angle as one float32 product.

    factor[i], llama3 rule (crates/model-format/src/mlx/config.rs:174-194):
    wavelen = 2 pi theta^(2i/R); below original/high -> 1; above original/low
    -> factor; between, smooth = (original/wavelen - low)/(high - low) and
    1/((1-smooth)/factor + smooth). `linear`: scale = 1/factor (config.rs:166-172).

    `yarn`: pair i keeps its frequency where it makes more than `fast_turns` turns within `original`
    positions, has it divided by `factor` where it makes fewer than `slow_turns`, and a blend that is
    linear in i between: the (real) pair number that makes t turns is R ln(original / (2 pi t)) /
    (2 ln theta). Cosines and sines are then multiplied by `magnitude` = 0.1 ln(factor) + 1, which only
    the kernels of shaped attention layers apply (`rotary_table` refuses).

    Pairing (attention.metal:14-16): split-half rotates dimension i with i + R/2; adjacent
    rotates 2i with 2i + 1 (config key rope_traditional). The kernels rotate split-half; for
    adjacent pairs the mixer reorders each head's query and key rows once (even dimensions of
    the rotary part first, then the odd ones), after which pair i is again (i, i + R/2) with
    the same frequency, and every score q.k is unchanged.
    """

    graph_safe = True

    def __init__(self, head_dim: int, rotary_dim: int, theta: float, scaling: str = "default",
                 factor: float = 1.0, low_freq_factor: float = 1.0, high_freq_factor: float = 4.0,
                 original_max_position_embeddings: int = 0, adjacent_pairs: bool = False,
                 fast_turns: float = 32.0, slow_turns: float = 1.0):
        if rotary_dim <= 0 or rotary_dim > head_dim or rotary_dim % 2:
            raise InvalidError("rotary width must be even and at most the head size")
        if theta <= 0:
            raise InvalidError("rope theta must be positive")
        if scaling not in ("default", "linear", "llama3", "yarn"):
            raise UnsupportedError(f"RoPE type {scaling}")
        self.head_dim, self.rotary_dim, self.theta = head_dim, rotary_dim, float(theta)
        self.scaling, self.factor = scaling, float(factor)
        self.low, self.high = float(low_freq_factor), float(high_freq_factor)
        self.original = original_max_position_embeddings
        self.adjacent_pairs = bool(adjacent_pairs)
        self.fast_turns, self.slow_turns = float(fast_turns), float(slow_turns)
        self.magnitude = 1.0
        if scaling == "yarn":
            if self.factor <= 0 or self.original <= 0 or self.fast_turns <= 0 or self.slow_turns <= 0 or self.theta == 1.0:
                raise InvalidError("yarn scaling: factor, original positions and turns must be positive, theta not 1")
            self.magnitude = 0.1 * math.log(self.factor) + 1.0
        self.inv_freq: Optional[torch.Tensor] = None
        self.inv_freq64: Optional[torch.Tensor] = None

    def inverse_frequencies(self) -> List[float]:
        out = []
        R = self.rotary_dim
        low, high = self._yarn_range() if self.scaling == "yarn" else (0, 0)
        for i in range(R // 2):
            freq = self.theta ** (-2.0 * i / R)
            if self.scaling == "linear":
                freq *= 1.0 / self.factor
            elif self.scaling == "llama3":
                wavelen = 2.0 * math.pi * self.theta ** (2.0 * i / R)
                if wavelen < self.original / self.high:
                    divisor = 1.0
                elif wavelen > self.original / self.low:
                    divisor = self.factor
                else:
                    smooth = (self.original / wavelen - self.low) / (self.high - self.low)
                    divisor = 1.0 / ((1.0 - smooth) / self.factor + smooth)
                freq /= divisor
            elif self.scaling == "yarn":
                ramp = min(max((i - low) / max(high - low, 0.001), 0.0), 1.0)
                freq = freq / self.factor * ramp + freq * (1.0 - ramp)
            out.append(freq)
        return out

    def _yarn_range(self) -> Tuple[int, int]:
        """The pair numbers between which frequencies go over from kept to divided."""
        def pair_of(turns: float) -> float:
            return self.rotary_dim * math.log(self.original / (2.0 * math.pi * turns)) / (2.0 * math.log(self.theta))
        return max(math.floor(pair_of(self.fast_turns)), 0), min(math.ceil(pair_of(self.slow_turns)), self.rotary_dim - 1)

    def bind(self, weights, runtime) -> None:
        # layers with the same frequencies share one tensor, so that what is derived from it once
        # per step (a table of cosines and sines) serves them all
        frequencies = tuple(self.inverse_frequencies())
        key = (str(runtime.device), frequencies)
        if key not in _shared_frequencies:
            exact = torch.tensor(frequencies, dtype=torch.float64)
            # beside them in double precision, for kernels that form the angle in double precision
            _shared_frequencies[key] = (exact.to(torch.float32).to(runtime.device), exact.to(runtime.device))
        self.inv_freq, self.inv_freq64 = _shared_frequencies[key]

    def head_permutation(self) -> Optional[List[int]]:
        if not self.adjacent_pairs:
            return None
        R = self.rotary_dim
        return list(range(0, R, 2)) + list(range(1, R, 2)) + list(range(R, self.head_dim))

    def rotary_table(self) -> Optional[Tuple[torch.Tensor, int]]:
        if self.magnitude != 1.0:
            raise UnsupportedError("a rotation with a magnitude is built for shaped attention layers only")
        return self.inv_freq, self.rotary_dim


@register_position_encoding("distance_penalty")
class DistancePenalty(PositionEncoding):
    """No rotation: a key n positions behind its query loses slope_h * n from its score, with
    slope_h = 2^(-span (h + 1) / heads) for query head h = 0 .. heads - 1 (`span` 8 gives slopes
    from 2^(-8/heads) down to 2^-8). The slopes are made once, in double precision, and rounded
    to float32; the attention kernels subtract slope * float(distance) from the scaled score."""

    graph_safe = True

    def __init__(self, num_heads: int, span: float = 8.0):
        if num_heads <= 0 or span <= 0:
            raise InvalidError("a distance penalty needs heads and a positive span")
        self.num_heads, self.span = int(num_heads), float(span)
        self.slopes: Optional[torch.Tensor] = None

    def slope_values(self) -> List[float]:
        return [2.0 ** (-self.span * (h + 1) / self.num_heads) for h in range(self.num_heads)]

    def bind(self, weights, runtime) -> None:
        self.slopes = torch.tensor(self.slope_values(), dtype=torch.float64).to(torch.float32).to(runtime.device)

    def distance_slopes(self) -> Optional[torch.Tensor]:
        return self.slopes
