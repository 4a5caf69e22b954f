"""Rotary position encoding: f_i = theta^(-2i/n_rot) * scale computed in float64 and cast to
float32 (src/rope.zig:8-16); the angle float32(pos) * f_i and its cos/sin are computed inside
the q/k kernel (src/rope.zig:34-45); NeoX pairing (i, i + n_rot/2) unless `interleaved`
(src/rope.zig:50-64; NeoX for every architecture but llama, src/model.zig:449).

`yarn` = (factor, original, fast, slow): frequencies scaled for sequences longer than the `original` positions (YaRN; Peng et
al., "YaRN: Efficient Context Window Extension of Large Language Models").  A pair that turns more than `fast` times within the
original length keeps its frequency, one that turns less than `slow` times has it divided by `factor`, pairs between are
blended linearly in their index; cosines and sines are multiplied by 0.1 ln(factor) + 1."""
from __future__ import annotations

import math
from typing import Optional

import numpy as np
import torch

from .base import POSITION_ENCODINGS, PositionEncoding, RotaryParams


class RotaryEncoding(PositionEncoding):
    def __init__(self, head_dim: int, theta: float, n_rot: int | None = None, interleaved: bool = False,
                 scale: float = 1.0, yarn: Optional[tuple[float, float, float, float]] = None):
        self.head_dim = head_dim
        self.n_rot = head_dim if n_rot is None else n_rot
        if self.n_rot % 2 or self.n_rot > head_dim:
            raise ValueError(f"rotary width {self.n_rot} must be even and <= head_dim {head_dim}")   # src/model.zig:488-489
        self.theta, self.interleaved, self.scale = float(theta), interleaved, float(scale)
        if yarn is not None and (not yarn[0] > 0 or not yarn[1] > 0 or not yarn[2] > 0 or not yarn[3] > 0 or not theta > 1):
            raise ValueError(f"scaled rotation {yarn}: factor, original length and turns must be positive, the base above 1")
        self.yarn = None if yarn is None else tuple(float(v) for v in yarn)
        self._params: RotaryParams | None = None

    @property
    def amplitude(self) -> float:
        return 1.0 if self.yarn is None else 0.1 * math.log(self.yarn[0]) + 1.0

    def inv_freq_host(self) -> np.ndarray:
        i = np.arange(self.n_rot // 2, dtype=np.float64)
        f = np.power(np.float64(self.theta), -2.0 * i / np.float64(self.n_rot)) * self.scale
        if self.yarn is not None:
            factor, original, fast, slow = self.yarn

            def pair_of(turns):           # the (fractional) pair that turns so often within the original length
                return self.n_rot * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(self.theta))

            lo, hi = max(math.floor(pair_of(fast)), 0), min(math.ceil(pair_of(slow)), self.n_rot - 1)
            ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
            f = f / factor * ramp + f * (1.0 - ramp)
        return f.astype(np.float32)

    def load(self, weights, dtype, device):
        self._params = RotaryParams(torch.from_numpy(self.inv_freq_host()).to(device), self.n_rot, self.interleaved,
                                    self.amplitude)

    def rotary(self):
        return self._params


POSITION_ENCODINGS.register("rotary", RotaryEncoding)
