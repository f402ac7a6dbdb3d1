"""Position-encoding parts. A position part never touches activations itself: it hands the
mixer the constants that the kernels need, a rotation table and/or per-head score slopes.

Rotary: ``inv_freq_i = theta^(-2i/dim)`` in float32, divided by ``factor`` for linear scaling
(src/transformers/modeling_rope_utils.py:67, 100-108); pairs ``(i, i + dim/2)`` are rotated by
``position * inv_freq_i`` (src/transformers/models/falcon/modeling_falcon.py:76-108, 155-164).
ALiBi: per-head slopes of build_alibi_tensor (modeling_falcon.py:175-188), rounded to bfloat16
because the reference forms ``slope * position`` in bfloat16 (:196-197); the kernels round the
position and the product the same way.
"""
from __future__ import annotations

import math

import torch

from .base import BuildContext, Part, PartSpec, register_part


@register_part("position", "none")
class NoPosition(Part):
    graph_safe = True
    def __init__(self, build: BuildContext, spec: PartSpec):
        super().__init__(build, spec)

    def rotation(self):
        return None

    def score_bias(self):
        return None


@register_part("position", "rotary")
class RotaryPosition(NoPosition):
    def __init__(self, build: BuildContext, spec: PartSpec, head_dim: int, theta: float, factor: float = 1.0,
                 rotary_dim: int = 0, interleaved: bool = False, yarn: dict = None, bands: dict = None):
        super().__init__(build, spec)
        # which dims make a rotated pair: (i, i + dim / 2), the reference's rotate_half, or (2 i, 2 i + 1)
        self.interleaved = bool(interleaved)
        dim = int(rotary_dim) if rotary_dim else int(head_dim)
        if dim % 2 or dim > head_dim or dim <= 0:
            raise ValueError(f"rotary_dim must be even and in 2..head_dim, got {dim} for head_dim {head_dim}")
        exponent = torch.arange(0, dim, 2, dtype=torch.int64).float() / dim
        inv_freq = 1.0 / (float(theta) ** exponent)
        if factor != 1.0:
            inv_freq = inv_freq / float(factor)
        self.table_scale = 1.0
        if yarn:
            inv_freq, self.table_scale = yarn_frequencies(dim, float(theta), **yarn)
        if bands:
            inv_freq = banded_frequencies(dim, float(theta), **bands)
        self.inv_freq = inv_freq.to(torch.float32).to(build.device)
        # layers whose rotation has the same constants share one table of angles per step
        self.rotation_key = ("rotary", dim, float(theta), float(factor), tuple(sorted((yarn or {}).items())),
                             tuple(sorted((bands or {}).items())))

    def rotation(self):
        return self.inv_freq


def yarn_frequencies(dims: int, base: float, factor: float, original: float, fast: float, slow: float):
    """YaRN: frequencies that turn often within the ``original`` context stay as they are, those that turn seldom are
    divided by ``factor``, with a linear ramp between. With d(t) = dims ln(original / (2 pi t)) / (2 ln base) the
    index at which a frequency makes t turns over the original context, the ramp runs from lo = max(floor(d(fast)), 0)
    to hi = min(ceil(d(slow)), dims - 1): r_i = clamp((i - lo) / max(hi - lo, 0.001), 0, 1) and
    f_i' = (f_i / factor) r_i + f_i (1 - r_i). Cosines and sines are multiplied by 0.1 ln(factor) + 1. Computed in
    float64; returns (frequencies [dims / 2], that multiplier)."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = float(base) ** (-2.0 * i / dims)

    def index_of(turns: float) -> float:
        return dims * math.log(float(original) / (2.0 * math.pi * float(turns))) / (2.0 * math.log(float(base)))

    lo = max(math.floor(index_of(fast)), 0)
    hi = min(math.ceil(index_of(slow)), dims - 1)
    ramp = torch.clamp((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / float(factor) * ramp + f * (1.0 - ramp), 0.1 * math.log(float(factor)) + 1.0


def banded_frequencies(dims: int, base: float, factor: float, low: float, high: float, original: float) -> torch.Tensor:
    """Frequencies scaled by their wavelength l = 2 pi / f (the scaling of Llama 3.1): kept where l < original / high, divided
    by ``factor`` where l > original / low, and in between (1 - s) f / factor + s f with
    s = (original / l - low) / (high - low). Computed in float64; [dims / 2]."""
    f = float(base) ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    turns = float(original) * f / (2.0 * math.pi)          # original / l
    s = (turns - float(low)) / (float(high) - float(low))
    mixed = (1.0 - s) * f / float(factor) + s * f
    return torch.where(turns > float(high), f, torch.where(turns < float(low), f / float(factor), mixed))


def alibi_slopes(heads: int) -> torch.Tensor:
    """float32 slopes: a geometric series for the largest power of two below ``heads``, and the
    odd powers of the next finer series for the remaining heads."""
    n = 2 ** math.floor(math.log2(heads))
    first = torch.tensor(2.0 ** (-(2.0 ** -(math.log2(n) - 3))), dtype=torch.float32)
    slopes = torch.pow(first, torch.arange(1, n + 1, dtype=torch.int32))
    if n != heads:
        finer = torch.tensor(2.0 ** (-(2.0 ** -(math.log2(2 * n) - 3))), dtype=torch.float32)
        extra = torch.arange(1, 1 + 2 * min(n, heads - n), 2, dtype=torch.int32)
        slopes = torch.cat([slopes, torch.pow(finer, extra)])
    return slopes


@register_part("position", "alibi")
class AlibiPosition(NoPosition):
    def __init__(self, build: BuildContext, spec: PartSpec, heads: int):
        super().__init__(build, spec)
        self.slopes = alibi_slopes(int(heads)).bfloat16().float().to(build.device)

    def score_bias(self):
        return self.slopes
