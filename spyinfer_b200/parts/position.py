"""Position encodings that a mixer applies to its queries and keys.

``rotary_half``: pairs ``(j, j + r)`` with ``r = rotary_dim / 2``, ``freq_j = theta^(-j/r)``,
``angle = position * freq_j``, all in 32-bit; spymaster2h/spyinfer
src/utils/constant_table.hpp:28-41 (table) and src/backends/cpu/cpu_operator.cpp:397-408
(rotation).  ``rotary_interleaved``: the same angles on the pairs ``(2j, 2j + 1)`` (the
rule the reference's doc/op.md:58-95 describes and its code does not use).  Both take an
optional ``frequency_scale`` (every frequency divided by it: positions stretched linearly)
or explicit ``inverse_frequencies`` (one per pair: any other frequency function), or a
``wavelength_scaling`` (``factor``, ``low``, ``high``, ``original``: with the wavelength
``l = 2 pi / f``, a frequency stays where ``l < original / high``, becomes ``f / factor`` where
``l > original / low``, and in between is ``(1 - s) f / factor + s f`` with
``s = (original / l - low) / (high - low)``), or a ``yarn_scaling`` (``factor``, ``original``,
``fast``, ``slow``: with ``place(n) = dims ln(original / (2 pi n)) / (2 ln theta)``, the pair whose wavelength fits ``n`` times into
``original`` positions, ``lo = max(floor(place(fast)), 0)``, ``hi = min(ceil(place(slow)), dims - 1)`` and ``ramp_j`` rising from 0 at ``lo``
to 1 at ``hi``, a frequency becomes ``f / factor * ramp + f * (1 - ramp)``, and cos and sin are multiplied by ``0.1 ln(factor) + 1``), so a
scaled rotary encoding is a parameter, not a new kernel.  ``no_position``: nothing is applied.
"""
from __future__ import annotations

import math

import torch

from .. import kernels
from .base import PositionEncoding
from .registry import register_part

_TABLES = {}


@register_part("rotary_half")
class RotaryHalf(PositionEncoding):
    graph_safe = True
    """params: ``theta``, ``rotary_dim`` (even, at most the head size); optional
    ``frequency_scale`` (default 1), ``inverse_frequencies`` (a list of ``rotary_dim / 2``
    numbers that replaces ``theta^(-j/r)``) and ``wavelength_scaling`` (see the module's header;
    with it the frequencies are worked out in 64-bit and rounded once)."""

    def modules(self):
        return ["qk_rope_store"] + (["swiglu"] if self.magnitude != 1.0 else [])

    def __init__(self, params, ctx):
        super().__init__(params, ctx)
        self.theta, self.rotary_dim = float(params["theta"]), int(params["rotary_dim"])
        if self.rotary_dim <= 0 or self.rotary_dim % 2:
            raise ValueError(f"rotary_dim must be a positive even number, found {self.rotary_dim}")
        self.frequency_scale = float(params.get("frequency_scale", 1.0))
        if not self.frequency_scale > 0.0:
            raise ValueError(f"frequency_scale must be positive, found {self.frequency_scale}")
        self.given = params.get("inverse_frequencies")
        if self.given is not None and len(self.given) != self.rotary_dim // 2:
            raise ValueError(f"inverse_frequencies must name {self.rotary_dim // 2} frequencies, found {len(self.given)}")
        self.bands = params.get("wavelength_scaling")
        if self.bands is not None:
            b = {k: float(self.bands[k]) for k in ("factor", "low", "high", "original")}
            if not (b["factor"] > 0.0 and b["original"] > 0.0 and b["high"] > b["low"] > 0.0):
                raise ValueError(f"wavelength_scaling needs factor > 0, original > 0 and high > low > 0, found {self.bands}")
            self.bands = b
        self.yarn = params.get("yarn_scaling")
        if self.yarn is not None:
            y = {k: float(self.yarn[k]) for k in ("factor", "original", "fast", "slow")}
            if self.bands is not None or self.given is not None or min(y.values()) <= 0.0 or not self.theta > 1.0:
                raise ValueError(f"yarn_scaling needs positive factor, original, fast and slow, a base above 1 and no other scaling, found {self.yarn}")
            self.yarn = y

    @property
    def magnitude(self) -> float:
        """What cos and sin are multiplied by."""
        return 0.1 * math.log(self.yarn["factor"]) + 1.0 if self.yarn is not None else 1.0

    def _yarn_frequencies(self):
        y, dims = self.yarn, self.rotary_dim

        def place(turns):
            return dims * math.log(y["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(self.theta))

        lo, hi = max(math.floor(place(y["fast"])), 0), min(math.ceil(place(y["slow"])), dims - 1)
        out = []
        for j in range(dims // 2):
            f = self.theta ** (-2.0 * j / dims)
            ramp = min(max((j - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            out.append(f / y["factor"] * ramp + f * (1.0 - ramp))
        return out

    def inverse_frequencies(self) -> torch.Tensor:
        r = self.rotary_dim // 2
        if self.yarn is not None:
            inv = torch.tensor(self._yarn_frequencies(), dtype=torch.float64).to(torch.float32)
        elif self.bands is not None:
            b, out = self.bands, []
            base = [float(f) for f in self.given] if self.given is not None else [self.theta ** (-j / float(r)) for j in range(r)]
            for f in base:
                wave = 2.0 * math.pi / f
                if wave < b["original"] / b["high"]:
                    out.append(f)
                elif wave > b["original"] / b["low"]:
                    out.append(f / b["factor"])
                else:
                    s = (b["original"] / wave - b["low"]) / (b["high"] - b["low"])
                    out.append((1.0 - s) * f / b["factor"] + s * f)
            inv = torch.tensor(out, dtype=torch.float64).to(torch.float32)
        elif self.given is not None:
            inv = torch.tensor([float(f) for f in self.given], dtype=torch.float32)
        else:
            j = torch.arange(r, dtype=torch.float32)
            inv = torch.pow(torch.tensor(self.theta, dtype=torch.float32), -j / float(r))
        return inv / self.frequency_scale if self.frequency_scale != 1.0 else inv

    def rotation_table(self):
        key = (self.theta, self.rotary_dim, self.frequency_scale, tuple(self.given) if self.given is not None else None,
               tuple(sorted(self.bands.items())) if self.bands is not None else None, tuple(sorted(self.yarn.items())) if self.yarn is not None else None,
               self.ctx.max_model_len, str(self.ctx.device))
        if key not in _TABLES:
            inv = self.inverse_frequencies().to(self.ctx.device)
            table = kernels.build_rope_table(inv, self.ctx.max_model_len)
            _TABLES[key] = kernels.scale_(table, self.magnitude) if self.magnitude != 1.0 else table
        return _TABLES[key]


@register_part("rotary_interleaved")
class RotaryInterleaved(RotaryHalf):
    """As ``rotary_half`` with the pairs ``(2j, 2j + 1)``."""

    pairing = "interleaved"


@register_part("no_position")
class NoPosition(PositionEncoding):
    graph_safe = True
    pass
