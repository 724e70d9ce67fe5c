"""Rotary position encodings: plain RoPE, LongRoPE, YaRN and Llama 3.1's scaling, as frequency tables a mixer applies.

Parity with InfiniLM: `csrc/layers/rotary_embedding/rotary_embedding.cpp:50-113` (one rotary
object from head_dim, rotary_dim, max positions, theta, scaling), `rope_scaling_creators.cpp:23-47`
(LongRoPE takes short_factor, long_factor, original_max_position_embeddings, factor),
`csrc/config/model_config.hpp:139` (rotate-half pairing). The table arithmetic itself is inside
InfiniCore; here it is
    inv_freq[i] = 1 / (f[i] * theta^(2i/rot_dim)),  angle = position * inv_freq[i]
with f = 1 for plain RoPE. For LongRoPE, f is `long_factor` when the model's
max_position_embeddings exceeds original_max_position_embeddings, else `short_factor`, and
cos/sin are multiplied by sqrt(1 + ln(s) / ln(original_max)) with s = max/original (or `factor`
when given and not 1) if s > 1. The choice depends on the configuration only, never on the
length of the sequence at hand, so a position's encoding is the same however the work is cut.

YaRN (Peng, Quesnelle, Fan, Shippole: "YaRN: Efficient Context Window Extension of Large Language Models") divides by `factor`
the frequencies that turn fewer than `slow` times over the original length, keeps those that turn more than `fast` times,
blends linearly between, and multiplies cosine and sine by 0.1 ln(factor) + 1.

"llama3" (the scaling of Llama 3.1's rotary frequencies) also divides the slow ones by `factor` - those that turn fewer than `low`
times over the original length - and keeps those that turn more than `high` times; between, the two are blended linearly in the
number of turns, and cosine and sine stay as they are.
"""
from __future__ import annotations

import math
from typing import List, Optional

import torch

from .base import PositionEncoding, register_part


def rotary_inv_freq(rot_dim: int, theta: float, factors: Optional[List[float]]) -> List[float]:
    half = rot_dim // 2
    out = []
    for i in range(half):
        f = 1.0 if factors is None else float(factors[i])
        out.append(1.0 / (f * (float(theta) ** (2.0 * i / rot_dim))))
    return out


def longrope_choice(short_factor, long_factor, original_max: int, max_pos: int, factor: Optional[float]):
    """(factors, mscale) of a LongRoPE configuration."""
    s = max_pos / float(original_max)
    if factor is not None and factor != 1.0:
        s = float(factor)
    factors = long_factor if max_pos > original_max else short_factor
    mscale = math.sqrt(1.0 + math.log(s) / math.log(original_max)) if s > 1.0 else 1.0
    return factors, mscale


def yarn_inv_freq(rot_dim: int, theta: float, factor: float, original: float, fast: float, slow: float) -> List[float]:
    def dim_of(turns: float) -> float:            # the (real-valued) index whose wavelength fits `original` that many times
        return rot_dim * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(theta))
    lo = max(math.floor(dim_of(fast)), 0)
    hi = min(math.ceil(dim_of(slow)), rot_dim - 1)
    out = []
    for i, f in enumerate(rotary_inv_freq(rot_dim, theta, None)):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out


class Rope(PositionEncoding):
    """params: rot_dim, theta, interleaved (default False: dimension i pairs with i + rot_dim / 2)."""

    def __init__(self, params, prefix, dtype):
        super().__init__(params, prefix, dtype)
        self.rot_dim = int(params["rot_dim"])
        self.theta = float(params["theta"])
        self.mscale = 1.0
        self.interleaved = bool(params.get("interleaved", False))
        self._table = rotary_inv_freq(self.rot_dim, self.theta, None)
        self.inv_freq = None

    def to_device(self, device):
        self.freq64 = torch.tensor(self._table, dtype=torch.float64).to(device)
        self.inv_freq = self.freq64.to(torch.float32)


class LongRope(Rope):
    """params: rot_dim, theta, short_factor, long_factor, original_max_position_embeddings,
    max_position_embeddings, factor (optional)."""

    def __init__(self, params, prefix, dtype):
        PositionEncoding.__init__(self, params, prefix, dtype)
        self.rot_dim = int(params["rot_dim"])
        self.theta = float(params["theta"])
        factors, self.mscale = longrope_choice(params["short_factor"], params["long_factor"],
                                               int(params["original_max_position_embeddings"]),
                                               int(params["max_position_embeddings"]), params.get("factor"))
        if len(factors) != self.rot_dim // 2:
            raise ValueError("longrope: factor list must have rot_dim/2 entries")
        self._table = rotary_inv_freq(self.rot_dim, self.theta, factors)
        self.inv_freq = None


class YarnRope(Rope):
    """params: rot_dim, theta, interleaved, factor, original (positions), fast, slow (turns over them)."""

    def __init__(self, params, prefix, dtype):
        super().__init__(params, prefix, dtype)
        factor, original = float(params["factor"]), float(params["original"])
        fast, slow = float(params["fast"]), float(params["slow"])
        if min(factor, original, fast, slow) <= 0.0 or self.theta <= 0.0 or self.theta == 1.0:
            raise ValueError("yarn: factor, original, fast, slow must be positive, theta positive and not 1")
        self._table = yarn_inv_freq(self.rot_dim, self.theta, factor, original, fast, slow)
        self.mscale = 0.1 * math.log(factor) + 1.0


def llama3_inv_freq(rot_dim: int, theta: float, factor: float, original: float, low: float, high: float) -> List[float]:
    out = []
    for f in rotary_inv_freq(rot_dim, theta, None):
        turns = original * f / (2.0 * math.pi)
        if turns < low:
            f = f / factor
        elif turns <= high:
            keep = (turns - low) / (high - low)
            f = (1.0 - keep) * f / factor + keep * f
        out.append(f)
    return out


class Llama3Rope(Rope):
    """params: rot_dim, theta, interleaved, factor, original (positions), low, high (turns over them)."""

    def __init__(self, params, prefix, dtype):
        super().__init__(params, prefix, dtype)
        factor, original = float(params["factor"]), float(params["original"])
        low, high = float(params["low"]), float(params["high"])
        if min(factor, original) <= 0.0 or not low < high:
            raise ValueError("llama3: factor and original must be positive, low below high")
        self._table = llama3_inv_freq(self.rot_dim, self.theta, factor, original, low, high)


class NoPosition(PositionEncoding):
    """No position encoding (rot_dim 0)."""

    def __init__(self, params, prefix, dtype):
        super().__init__(params, prefix, dtype)
        self.rot_dim, self.mscale, self.inv_freq = 0, 1.0, None


register_part("position", "rope", Rope)
register_part("position", "longrope", LongRope)
register_part("position", "yarn", YarnRope)
register_part("position", "llama3", Llama3Rope)
register_part("position", "none", NoPosition)
