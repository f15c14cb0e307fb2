"""Rotary position encoding, half-split (NeoX) pairing unless the spec's `pairing`
parameter says "consecutive".

For a head vector t[0..d) and i < rd/2:  theta = (float)pos / base^(2i/rd);
(t_i, t_{i+rd/2}) <- (t_i cos - t_{i+rd/2} sin, t_i sin + t_{i+rd/2} cos);
elements >= rd stay (src/kernels_cuda/rope.cu:9-37).  The part owns the table
of denominators base^(2i/rd), made once on the host in double precision and
rounded to 32-bit; the angle itself is computed per element in 32-bit inside
the fused kernel that the attention part launches.  Pairing and magnitude go
to that kernel as parameters (`Rotation`), so an encoding with consecutive
pairs or a scaled magnitude is another position part, not another kernel.
"""

from __future__ import annotations

import math
from typing import Dict, Optional, Tuple

import torch

from ..config.spec import PositionSpec
from ..errors import InvalidInput
from .registry import Rotation, TensorInfo, register_position


@register_position("rope_neox")
class RotaryNeox:
    capturable = True
    magnitude = 1.0  # of the cosines and sines

    def __init__(self, spec: PositionSpec, dtype: torch.dtype, device):
        if spec.rotary_dim % 2 or not (0 < spec.rotary_dim <= spec.head_dim):
            raise InvalidInput(
                f"rotary_dim must be even and in (0, head_dim], got {spec.rotary_dim}"
            )
        self.spec = spec
        half = spec.rotary_dim // 2
        # the C library's pow in double, element by element, then one rounding to 32-bit
        denom = [math.pow(float(spec.theta), 2.0 * i / float(spec.rotary_dim)) for i in range(half)]
        self.denominators = torch.tensor(denom, dtype=torch.float64).to(torch.float32).to(device)

    @classmethod
    def tensor_specs(cls, spec: PositionSpec) -> Dict[str, TensorInfo]:
        return {}

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        pass

    def rotation(self) -> Rotation:
        pairing = str(dict(self.spec.params).get("pairing", "half"))
        return Rotation(self.denominators, self.spec.rotary_dim, pairing, self.magnitude)


@register_position("rope_linear")
class RotaryLinear(RotaryNeox):
    """The half-split rotation with every frequency divided by the parameter `factor`:
    the pair turns by position / (factor * theta^(2i/rd)).  Only the table of
    denominators differs from the plain encoding."""

    def __init__(self, spec: PositionSpec, dtype: torch.dtype, device):
        super().__init__(spec, dtype, device)
        factor = float(dict(spec.params).get("factor", 1.0))
        if not factor > 0:
            raise InvalidInput("rope_linear: factor must be positive")
        denom = [factor * math.pow(float(spec.theta), 2.0 * i / float(spec.rotary_dim))
                 for i in range(spec.rotary_dim // 2)]
        self.denominators = torch.tensor(denom, dtype=torch.float64).to(torch.float32).to(device)


@register_position("rope_scaled")
class RotaryScaled(RotaryNeox):
    """The half-split rotation with wavelength-dependent frequency scaling.

    With f_i = theta^(-2i/rd) and the wavelength l = 2 pi / f_i, and the
    parameters `factor`, `low`, `high`, `original`: f_i stays where
    l < original / high; becomes f_i / factor where l > original / low; and in
    between, with s = (original / l - low) / (high - low), the blend
    (1 - s) f_i / factor + s f_i.  Only the table of denominators (1 / f_i)
    differs from the plain encoding."""

    def __init__(self, spec: PositionSpec, dtype: torch.dtype, device):
        super().__init__(spec, dtype, device)
        p = dict(spec.params)
        factor, low, high, original = (float(p[k]) for k in ("factor", "low", "high", "original"))
        if factor <= 0 or high <= low or original <= 0:
            raise InvalidInput("rope_scaled: factor and original must be positive and high above low")
        half = spec.rotary_dim // 2
        denom = []
        for i in range(half):
            f = math.pow(float(spec.theta), -2.0 * i / float(spec.rotary_dim))
            wave = 2.0 * math.pi / f
            if wave < original / high:
                g = f
            elif wave > original / low:
                g = f / factor
            else:
                s = (original / wave - low) / (high - low)
                g = (1.0 - s) * f / factor + s * f
            denom.append(1.0 / g)
        self.denominators = torch.tensor(denom, dtype=torch.float64).to(torch.float32).to(device)


@register_position("rope_yarn")
class RotaryYarn(RotaryNeox):
    """The rotation with frequencies scaled by how often a pair turns within the
    original context, and a magnitude.

    A pair i of plain frequency g_i = theta^(-2i/rd) makes N g_i / (2 pi) turns within
    N = `original` positions; the pair that makes t of them has the fractional index
    j(t) = rd / 2 * log_theta(N / (2 pi t)).  Pairs up to a = floor(j(`fast`)) (at
    least 0) keep g_i, pairs from b = ceil(j(`slow`)) (at most rd - 1) on turn `factor`
    times slower, and between them the two frequencies are blended with the weight
    s_i = (i - a) / (b - a) on the slower one (the width b - a taken as 0.001 at least,
    s_i kept within 0 and 1).  Cosine and sine grow by 1 + ln(factor) / 10."""

    def __init__(self, spec: PositionSpec, dtype: torch.dtype, device):
        super().__init__(spec, dtype, device)
        p = dict(spec.params)
        factor, original, fast, slow = (float(p[k]) for k in ("factor", "original", "fast", "slow"))
        if min(factor, original, fast, slow) <= 0 or spec.theta <= 0 or spec.theta == 1:
            raise InvalidInput("rope_yarn: factor, original, fast and slow must be positive, theta positive and not 1")
        rd, base = spec.rotary_dim, float(spec.theta)

        def index_of(turns: float) -> float:
            return rd * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

        first, last = max(math.floor(index_of(fast)), 0), min(math.ceil(index_of(slow)), rd - 1)
        denom = []
        for i in range(rd // 2):
            g = math.pow(base, -2.0 * i / float(rd))
            s = min(max((i - first) / max(last - first, 0.001), 0.0), 1.0)
            denom.append(1.0 / (g / factor * s + g * (1.0 - s)))
        self.denominators = torch.tensor(denom, dtype=torch.float64).to(torch.float32).to(device)
        self.magnitude = 0.1 * math.log(factor) + 1.0
