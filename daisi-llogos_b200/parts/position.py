"""Position encodings.

``RotaryEncoding`` owns the cos/sin tables of rotary position encoding.  Frequencies
and angles are computed in float64 on the host, as the reference does
(Daisi.Llogos.Cpu/Rope.cs:131-162: ``freq_i = 1 / theta^(2i/rotary_dim)``,
``angle = position * freq_i``), and stored as float32.  The rotation itself happens
inside the mixer's fused query/key kernel; ``pairing`` says which elements form a
pair: "half" pairs ``(i, i + rotary_dim/2)`` (Rope.cs:42-63, the layout of
safetensors checkpoints), "adjacent" pairs ``(2i, 2i+1)`` (Rope.cs:150-161, the layout
of converted GGUF files).
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional

import torch

from .base import PositionEncoding, register_part


@dataclass
class Rotation:
    cos: torch.Tensor        # [positions, rotary_dim / 2] float32, on the device
    sin: torch.Tensor
    rotary_dim: int
    pairing: int             # 0 = half, 1 = adjacent


def rotary_amplitude(scaling: Optional[dict]) -> float:
    """What cos and sin are multiplied by: 1, or for yarn scaling ``amplitude_slope * ln(factor) + 1``."""
    if scaling and scaling.get("rope_type") == "yarn":
        return float(scaling.get("amplitude_slope", 0.1)) * math.log(float(scaling["factor"])) + 1.0
    return 1.0


def rotary_inverse_frequencies(rotary_dim: int, theta: float, scaling: Optional[dict]) -> torch.Tensor:
    """float64 ``[rotary_dim / 2]``; ``scaling`` is a llama3 or yarn ``rope_scaling`` dict or None.

    yarn: pair i makes ``t_i = L f_i / (2 pi)`` turns over the original context ``L``; the pair index at which a
    frequency makes ``t`` turns is ``d(t) = rotary_dim ln(L / (2 pi t)) / (2 ln theta)``.  With ``lo = max(floor(d(beta_fast)),
    0)`` and ``hi = min(ceil(d(beta_slow)), rotary_dim - 1)`` the ramp ``r_i = clamp((i - lo) / max(hi - lo, 0.001), 0, 1)``
    blends ``f' = r f / factor + (1 - r) f``: fast pairs keep their frequency, slow ones are stretched by ``factor``.
    (The amplitude that goes with it is ``rotary_amplitude``.)

    llama3: with wavelength ``lam = 2 pi / f`` and ``L`` the original context length,
    ``f`` is kept where ``lam < L / high_freq_factor``, divided by ``factor`` where
    ``lam > L / low_freq_factor``, and interpolated between:
    ``s = (L / lam - low) / (high - low)``, ``f' = (1 - s) f / factor + s f``.
    """
    half = rotary_dim // 2
    i = torch.arange(half, dtype=torch.float64)
    inv = 1.0 / torch.pow(torch.tensor(float(theta), dtype=torch.float64), 2.0 * i / rotary_dim)
    if scaling and scaling.get("rope_type") == "yarn":
        factor = float(scaling["factor"])
        orig = float(scaling["original_max_position_embeddings"])

        def pair_of(turns: float) -> float:
            return rotary_dim * math.log(orig / (2.0 * math.pi * turns)) / (2.0 * math.log(float(theta)))

        lo = max(math.floor(pair_of(float(scaling["beta_fast"]))), 0)
        hi = min(math.ceil(pair_of(float(scaling["beta_slow"]))), rotary_dim - 1)
        ramp = torch.clamp((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
        return inv / factor * ramp + inv * (1.0 - ramp)
    if scaling:
        if scaling.get("rope_type") != "llama3":
            raise ValueError(f"rotary scaling '{scaling.get('rope_type')}' is not supported")
        factor = float(scaling["factor"])
        low = float(scaling["low_freq_factor"])
        high = float(scaling["high_freq_factor"])
        orig = float(scaling["original_max_position_embeddings"])
        lam = 2.0 * math.pi / inv
        smooth = (orig / lam - low) / (high - low)
        mid = (1.0 - smooth) * inv / factor + smooth * inv
        inv = torch.where(lam < orig / high, inv, torch.where(lam > orig / low, inv / factor, mid))
    return inv


class RotaryEncoding(PositionEncoding):
    """params: head_dim, rotary_dim (<= head_dim, even), theta, scaling (dict or None), pairing."""

    def __init__(self, params, prefix, env):
        super().__init__(params, prefix, env)
        self.rotary_dim = int(params["rotary_dim"])
        if self.rotary_dim <= 0 or self.rotary_dim % 2 or self.rotary_dim > int(params["head_dim"]):
            raise ValueError(f"rotary_dim {self.rotary_dim} must be even and at most head_dim {params['head_dim']}")
        pairing = params.get("pairing", "half")
        if pairing not in ("half", "adjacent"):
            raise ValueError(f"rotary pairing '{pairing}' is not known (half, adjacent)")
        self.pairing = 0 if pairing == "half" else 1
        self._rotation: Optional[Rotation] = None
        self._retired = []        # smaller tables that were replaced: a recorded CUDA graph may still read them

    def limit(self) -> Optional[int]:
        return None if self._rotation is None else int(self._rotation.cos.shape[0])

    def prepare(self, max_positions: int) -> None:
        if self._rotation is not None:
            if self._rotation.cos.shape[0] >= max_positions:
                return
            self._retired.append(self._rotation)
        inv = rotary_inverse_frequencies(self.rotary_dim, self.params["theta"], self.params.get("scaling"))
        pos = torch.arange(max_positions, dtype=torch.float64)
        ang = pos[:, None] * inv[None, :]
        amp = rotary_amplitude(self.params.get("scaling"))
        cos = (amp * torch.cos(ang)).to(torch.float32).to(self.env.device).contiguous()
        sin = (amp * torch.sin(ang)).to(torch.float32).to(self.env.device).contiguous()
        self._rotation = Rotation(cos, sin, self.rotary_dim, self.pairing)

    def rotation(self) -> Rotation:
        if self._rotation is None:
            raise RuntimeError("RotaryEncoding.prepare() has not run")
        return self._rotation


class QueryTemperature(PositionEncoding):
    """Queries grow with their position: a query at position p is multiplied by ``1 + coef ln(floor((p + 1) / every) + 1)``.
    The factors are worked out in float64 and kept as float32, one per position.  params: coef, every."""

    def __init__(self, params, prefix, env):
        super().__init__(params, prefix, env)
        self.coef, self.every = float(params["coef"]), float(params["every"])
        if not self.every > 0:
            raise ValueError(f"query temperature: 'every' must be positive, got {self.every}")
        self._table: Optional[torch.Tensor] = None
        self._retired = []        # as in RotaryEncoding

    def limit(self) -> Optional[int]:
        return None if self._table is None else int(self._table.shape[0])

    def prepare(self, max_positions: int) -> None:
        if self._table is not None:
            if self._table.shape[0] >= max_positions:
                return
            self._retired.append(self._table)
        pos = torch.arange(max_positions, dtype=torch.float64)
        factor = 1.0 + self.coef * torch.log(torch.floor((pos + 1.0) / self.every) + 1.0)
        self._table = factor.to(torch.float32).to(self.env.device).contiguous()

    def query_scale(self) -> torch.Tensor:
        if self._table is None:
            raise RuntimeError("QueryTemperature.prepare() has not run")
        return self._table


class NoEncoding(PositionEncoding):
    """No position information (mixers then skip the rotation)."""


register_part("position", "rotary", RotaryEncoding)
register_part("position", "query_temperature", QueryTemperature)
register_part("position", "none", NoEncoding)
