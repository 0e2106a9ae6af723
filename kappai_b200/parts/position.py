"""Position encodings of a mixer.

``rope``: rotary encoding.  The angle table is built on the host in double
precision, ``angle = pos * theta^(-2j/rotary_dim)``, and stored as float32
cos/sin ``[max_positions, rotary_dim/2]`` (src/compute.c:22-65; the reference
shares one table between all layers with the same sizes, src/compute.c:80-102,
and so does this).  ``pairing`` is ``neox`` (j, j + rotary_dim/2) or
``interleaved`` (2j, 2j+1) (src/backend/cpu/scalar/core.c:66-84); ``rotary_dim``
may be smaller than the head size (the rest of the head is left as it is).
``scaling`` (optional; keys ``factor``, ``low``, ``high``, ``original``) rescales the
frequencies by their wavelength ``l = 2 pi / f``: a frequency with
``l < original / high`` is kept, one with ``l > original / low`` is divided by
``factor``, and between the two, with ``s = (original / l - low) / (high - low)``,
it becomes ``(1 - s) f / factor + s f``.  With the key ``factor`` alone every
frequency is divided by it.  With the keys ``factor``, ``original``, ``fast`` and
``slow`` (YaRN) the blend runs over the pairs instead: pair t(n) = dims ln(original
/ (2 pi n)) / (2 ln theta) turns n times over the original length, the pairs up
to floor(t(fast)) keep their frequency, those from ceil(t(slow)) on are divided
by ``factor``, linearly in between; and the cosines and sines are multiplied by
``0.1 ln(factor) + 1``.

``none``: no rotation.
"""
from __future__ import annotations

import numpy as np
import torch

from ..config.schema import ConfigError
from .base import Part, register_part


def scaled_frequencies(f: np.ndarray, scaling) -> np.ndarray:
    """Rotary frequencies rescaled by wavelength (see the module's text); ``scaling`` is
    (factor, low, high, original), (factor,), ("yarn", factor, original, fast, slow, theta) or None."""
    if scaling is None:
        return f
    if len(scaling) == 1:
        return f / scaling[0]
    if scaling[0] == "yarn":
        _, factor, original, fast, slow, theta = scaling
        dims = 2 * len(f)
        pair = lambda turns: dims * np.log(original / (2.0 * np.pi * turns)) / (2.0 * np.log(theta))
        lo, hi = max(np.floor(pair(fast)), 0.0), min(np.ceil(pair(slow)), dims - 1.0)
        ramp = np.clip((np.arange(len(f)) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
        return f / factor * ramp + f * (1.0 - ramp)
    factor, low, high, original = scaling
    lam = 2.0 * np.pi / f
    s = (original / lam - low) / (high - low)
    blend = (1.0 - s) * f / factor + s * f
    return np.where(lam < original / high, f, np.where(lam > original / low, f / factor, blend))


class RotaryEncoding(Part):
    category = "position"
    graph_safe = True

    def __init__(self, params, env):
        super().__init__(params, env)
        self.rotary_dim = int(self._p("rotary_dim"))
        self.theta = float(self._p("theta"))
        pairing = self._p("pairing", "neox")
        if pairing not in ("neox", "interleaved"):
            raise ConfigError(f"rope: pairing '{pairing}' (expected 'neox' or 'interleaved')")
        if self.rotary_dim < 2 or self.rotary_dim % 2:
            raise ConfigError(f"rope: rotary_dim={self.rotary_dim} must be even and positive")
        self.interleaved = pairing == "interleaved"
        scaling = self._p("scaling", None)
        self.scaling = None
        if scaling and set(scaling) == {"factor"}:
            self.scaling = (float(scaling["factor"]),)
            if not self.scaling[0] > 0:
                raise ConfigError("rope: scaling wants factor > 0")
        elif scaling and set(scaling) == {"factor", "original", "fast", "slow"}:
            self.scaling = ("yarn",) + tuple(float(scaling[k]) for k in ("factor", "original", "fast", "slow")) + (self.theta,)
            if min(self.scaling[1:5]) <= 0 or self.theta <= 0 or self.theta == 1.0:
                raise ConfigError("rope: scaling wants factor, original, fast and slow > 0")
        elif scaling:
            try:
                self.scaling = tuple(float(scaling[k]) for k in ("factor", "low", "high", "original"))
            except (KeyError, TypeError, ValueError):
                raise ConfigError("rope: scaling needs the numbers factor, low, high and original") from None
            factor, low, high, original = self.scaling
            if factor <= 0 or original <= 0 or low <= 0 or high <= low:
                raise ConfigError("rope: scaling wants factor, original, low > 0 and high > low")
        key = ("rope", self.rotary_dim, self.theta, self.scaling, env.max_positions)
        if key not in env.shared:
            half = self.rotary_dim // 2
            inv = scaled_frequencies(
                np.power(self.theta, -2.0 * np.arange(half, dtype=np.float64) / self.rotary_dim), self.scaling)
            ang = np.arange(env.max_positions, dtype=np.float64)[:, None] * inv[None, :]
            m = 0.1 * np.log(self.scaling[1]) + 1.0 if self.scaling and self.scaling[0] == "yarn" else 1.0
            env.shared[key] = (torch.from_numpy((np.cos(ang) * m).astype(np.float32)).to(env.device),
                               torch.from_numpy((np.sin(ang) * m).astype(np.float32)).to(env.device))
        self.cos, self.sin = env.shared[key]

    def fused_rotary(self):
        return self.cos, self.sin, self.rotary_dim, self.interleaved


class NoPosition(Part):
    category = "position"
    graph_safe = True

    def fused_rotary(self):
        return None, None, 0, False


register_part("position", "rope", RotaryEncoding)
register_part("position", "none", NoPosition)
