"""Position encodings.

``rope_neox``: partial NeoX rotary embedding.  ``inv_freq_i = 1 / theta^(2i / rotary_dim)``,
angle = ``float32(position) * inv_freq_i``, table ``cos || sin`` of shape
``[positions, rotary_dim]`` in float32 (python/freetoken/layers/rotary.py:49-59).  The table is
computed once on the host with the same float32 operations as the reference and uploaded,
so every consumer (and a CPU check) sees identical angles; it covers the engine's longest
sequence rather than the checkpoint's ``max_position_embeddings``.  Mixers rotate inside
their own kernels (``norm_rope_store``); one table serves all layers with equal parameters
(``get_rope`` is cached the same way, rotary.py:211-231).

``rope_interleaved``: the same angles and table; the pairs that turn together are the neighbours ``(2i, 2i + 1)``
instead of ``(i, i + rotary_dim / 2)``.  A mixer's kernel asks the part (``interleaved``) which pairing to use.

``yarn`` (a parameter of both): frequencies stretched for contexts longer than the ``original`` one a model was trained on
(YaRN).  With ``index(t) = rotary_dim ln(original / (2 pi t)) / (2 ln theta)``, the index whose pair turns ``t`` times over
the original context, ``lo = max(floor(index(fast)), 0)`` and ``hi = min(ceil(index(slow)), rotary_dim - 1)``, pair ``i``
turns at ``f_i / factor`` with the share ``ramp_i = clamp((i - lo) / max(hi - lo, 0.001), 0, 1)`` and at ``f_i`` with the
rest; cosines and sines are multiplied by ``0.1 ln(factor) + 1``.

``band_scaling`` (a parameter of both, as Llama 3.1 stretches its frequencies): ``(factor, low, high, original)``.  A pair whose
wavelength ``2 pi / f`` is shorter than ``original / high`` keeps ``f``, one longer than ``original / low`` turns at
``f / factor``, and in between the two are blended with ``s = (original f / (2 pi) - low) / (high - low)`` on ``f``.

``none``: no position encoding (a mixer that needs none asks for this kind).

``log_temperature``: no rotation; the table holds one factor per position,
``1 + coef * ln(floor((p + 1) / every) + 1)``, by which a mixer multiplies its queries, so that
attention sharpens as the context grows.  Computed in float64 on the host and rounded once to
float32.
"""

from __future__ import annotations

import math
from typing import Optional

import torch

from ..config.spec import PartSpec
from ..errors import ConfigError
from .base import POSITIONS, BuildEnv, PositionEncoding


@POSITIONS.register("rope_neox")
class NeoxRope(PositionEncoding):
    """params: ``rotary_dim`` (even, <= head_dim; 0 disables), ``theta``, ``precise`` (False: the reference's
    float32 operations; True: angles, cosines and sines in float64, rounded to float32 once), ``yarn`` (None, or
    ``(factor, original, fast, slow)``; needs ``precise``), ``band_scaling`` (None, or ``(factor, low, high, original)``; needs
    ``precise``; not with ``yarn``)."""

    interleaved = False

    def __init__(self, spec: PartSpec, env: BuildEnv):
        super().__init__(spec, env)
        self.rotary_dim = int(spec["rotary_dim"])
        self.theta = float(spec["theta"])
        if self.rotary_dim % 2 or self.rotary_dim < 0:
            raise ConfigError(f"rope_neox: rotary_dim={self.rotary_dim} must be even and >= 0")
        self.yarn = spec.get("yarn")
        if self.yarn is not None and not spec.get("precise", False):
            raise ConfigError("rope: stretched frequencies are computed in float64 (precise)")
        self.bands = spec.get("band_scaling")
        if self.bands is not None and (self.yarn is not None or not spec.get("precise", False)):
            raise ConfigError("rope: frequencies are scaled in one way, in float64 (precise)")
        self._table: Optional[torch.Tensor] = None

    def frequencies(self) -> torch.Tensor:
        """One per pair, float64."""
        rd = self.rotary_dim
        f = self.theta ** (-torch.arange(0, rd, 2, dtype=torch.float64) / rd)
        if self.bands is not None:
            factor, low, high, original = (float(x) for x in self.bands)
            wave = 2.0 * math.pi / f
            s = (original / wave - low) / (high - low) if high != low else torch.zeros_like(f)
            mixed = (1.0 - s) * f / factor + s * f
            return torch.where(wave < original / high, f, torch.where(wave > original / low, f / factor, mixed))
        if self.yarn is None:
            return f
        factor, original, fast, slow = (float(x) for x in self.yarn)

        def index(turns: float) -> float:
            return rd * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(self.theta))

        lo, hi = max(math.floor(index(fast)), 0), min(math.ceil(index(slow)), rd - 1)
        ramp = ((torch.arange(rd // 2, dtype=torch.float64) - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        return f / factor * ramp + f * (1.0 - ramp)

    def magnitude(self) -> float:
        """The factor on cosines and sines."""
        return 1.0 if self.yarn is None else 0.1 * math.log(float(self.yarn[0])) + 1.0

    def table(self) -> Optional[torch.Tensor]:
        """Built at the first call: by then the engine has settled its longest sequence
        (``env.max_seq_len`` may shrink between a part's construction and the first step, once
        the cache has been sized)."""
        if self._table is None and self.rotary_dim:
            rd = self.rotary_dim
            if self.spec.get("precise", False):
                ang = torch.arange(self.env.max_seq_len, dtype=torch.float64)[:, None] * self.frequencies()[None, :]
                tab = torch.cat((ang.cos(), ang.sin()), dim=-1) * self.magnitude()
                self._table = tab.float().contiguous().to(self.env.device)
                return self._table
            inv_freq = 1.0 / (self.theta ** (torch.arange(0, rd, 2, dtype=torch.float) / rd))
            t = torch.arange(self.env.max_seq_len, dtype=torch.float)
            freqs = torch.einsum("i,j -> ij", t, inv_freq)
            self._table = torch.cat((freqs.cos(), freqs.sin()), dim=-1).contiguous().to(self.env.device)
        return self._table


@POSITIONS.register("rope_interleaved")
class InterleavedRope(NeoxRope):
    """params: as ``rope_neox``.  Dimension ``2i`` turns with dimension ``2i + 1`` by ``position * theta^(-2i / rotary_dim)``."""

    interleaved = True


@POSITIONS.register("log_temperature")
class LogTemperature(PositionEncoding):
    """params: ``coef``, ``every`` (positive integer)."""

    rotary_dim = 0

    def __init__(self, spec: PartSpec, env: BuildEnv):
        super().__init__(spec, env)
        self.coef = float(spec["coef"])
        self.every = int(spec["every"])
        if self.every < 1:
            raise ConfigError(f"log_temperature: every={self.every} must be >= 1")
        self._table: Optional[torch.Tensor] = None

    def table(self) -> Optional[torch.Tensor]:
        return None  # nothing to rotate by

    def scale_table(self) -> torch.Tensor:
        """``[positions]`` float32 factors, built at the first call (see :meth:`NeoxRope.table`)."""
        if self._table is None:
            p = torch.arange(self.env.max_seq_len, dtype=torch.int64)
            steps = torch.div(p + 1, self.every, rounding_mode="floor") + 1
            self._table = (1.0 + self.coef * torch.log(steps.double())).float().contiguous().to(self.env.device)
        return self._table


@POSITIONS.register("none")
class NoPosition(PositionEncoding):
    rotary_dim = 0

    def table(self) -> Optional[torch.Tensor]:
        return None


def shared_position(spec: PartSpec, env: BuildEnv) -> PositionEncoding:
    """One instance per distinct spec for the whole model."""
    key = ("position", spec.key())
    if key not in env.shared:
        env.shared[key] = POSITIONS.build(spec, env)
    return env.shared[key]
