"""Rotary position encoding over the first ``rotary_dim`` elements of a head:
inv_freq_i = theta^(-2i/rotary_dim) / divide_by (divide_by 1 unless positions are scaled linearly), angle = position * inv_freq_i
(infer/src/weight_loader.rs:955-989).  ``pairing`` says which two elements turn
together: "half" pairs element i with i + rotary_dim/2 (Qwen3), "interleaved" pairs
element 2i with 2i + 1.  ``stretch`` (YaRN) makes a context ``factor`` times the original one out of the frequencies: with
pair(n) = rotary_dim * ln(original / (2 pi n)) / (2 ln theta) the pair that turns n times within the original context, pairs
below floor(pair(fast)) keep their frequency, pairs above ceil(pair(slow)) have it divided by the factor, a linear ramp
between, and cosines and sines are multiplied by 0.1 ln(factor) + 1 (``amplitude``).  The reference tabulates cos and
sin of every position in bfloat16; here the kernels evaluate sincosf of the float32
angle of the positions they meet (for prompt portions once per step, into a table
that the step's layers share), so there is no limit on the position."""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import ClassVar, Optional

import torch

from .base import PositionEncoding
from .registry import register_part


@dataclass(frozen=True)
class RotaryStretch:
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class RotarySpec:
    rotary_dim: int
    theta: float
    pairing: str = "half"
    divide_by: float = 1.0          # linear scaling of positions: every frequency is divided by this
    stretch: Optional[RotaryStretch] = None
    kind: ClassVar[str] = "rotary"


class Rotary(PositionEncoding):
    def __init__(self, spec: RotarySpec):
        if spec.rotary_dim <= 0 or spec.rotary_dim % 2:
            raise ValueError(f"rotary_dim must be positive and even, got {spec.rotary_dim}")
        if spec.pairing not in ("half", "interleaved"):
            raise ValueError(f"rotary pairing must be 'half' or 'interleaved', got {spec.pairing!r}")
        if not spec.divide_by > 0:
            raise ValueError(f"rotary divide_by must be positive, got {spec.divide_by}")
        if spec.stretch is not None and not (spec.stretch.factor > 0 and spec.stretch.original > 0 and spec.stretch.fast > 0
                                             and spec.stretch.slow > 0 and spec.theta > 1):
            raise ValueError(f"rotary stretch: factor, original, fast and slow must be positive and theta above 1, got {spec.stretch}")
        self.spec = spec
        self.inv_freq = None
        self.amplitude = 1.0 if spec.stretch is None else 0.1 * math.log(spec.stretch.factor) + 1.0

    def load(self, tensors, dtype, device):
        i = torch.arange(self.spec.rotary_dim // 2, dtype=torch.float64)
        inv = torch.pow(torch.tensor(self.spec.theta, dtype=torch.float64), -2.0 * i / self.spec.rotary_dim) / self.spec.divide_by
        st = self.spec.stretch
        if st is not None:
            lo, hi = (self.spec.rotary_dim * math.log(st.original / (2.0 * math.pi * n)) / (2.0 * math.log(self.spec.theta)) for n in (st.fast, st.slow))
            lo, hi = max(math.floor(lo), 0), min(math.ceil(hi), self.spec.rotary_dim - 1)
            ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
            inv = inv / st.factor * ramp + inv * (1.0 - ramp)
        self.inv_freq = inv.to(torch.float32).to(device)

    def rotary(self):
        return self.inv_freq, self.spec.rotary_dim

    @property
    def pairing(self) -> str:
        return self.spec.pairing


register_part(RotarySpec.kind, Rotary)
