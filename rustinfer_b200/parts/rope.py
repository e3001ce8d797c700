"""Rotary position encoding: the frequency law and the cos/sin tables.

inv_freq f_i = theta^(-2i/rotary_dim); with llama3 scaling each frequency is kept, divided
by `factor`, or blended, by the band its wavelength falls in
(crates/infer-worker/src/models/loader.rs:1543-1571).  Angles pos*f_i are formed in
float64 and the tables are stored fp32 [positions, rotary_dim/2]; RustInfer stores them in
the activation dtype (bf16 in production, :1574-1589), which costs three digits of the
angle for nothing.  The rotation itself (pair i, i+rotary_dim/2) is in the kernel that
also writes keys and values into the cache.
"""
from __future__ import annotations

import math
from typing import List, Optional

import torch

from .base import BuildContext, PositionEncoding, register_position


def rope_inv_freq(rotary_dim: int, theta: float, scaling: Optional[dict]) -> List[float]:
    half = rotary_dim // 2
    freqs = [theta ** (-2.0 * i / rotary_dim) for i in range(half)]
    if not scaling:
        return freqs
    kind = scaling.get("rope_type", scaling.get("type"))
    if kind not in ("llama3", "yarn"):
        raise ValueError(f"rope scaling of type {kind!r} is not built; known: 'llama3', 'yarn'")
    factor = float(scaling["factor"])
    orig = float(scaling["original_max_position_embeddings"])
    if kind == "yarn":
        def pair_turning(turns: float) -> float:
            return rotary_dim * math.log(orig / (2.0 * math.pi * turns)) / (2.0 * math.log(theta))
        lo = max(math.floor(pair_turning(float(scaling["beta_fast"]))), 0)
        hi = min(math.ceil(pair_turning(float(scaling["beta_slow"]))), rotary_dim - 1)
        for i, f in enumerate(freqs):
            ramp = min(1.0, max(0.0, (i - lo) / max(hi - lo, 0.001)))
            freqs[i] = f / factor * ramp + f * (1.0 - ramp)
        return freqs
    low = float(scaling["low_freq_factor"])
    high = float(scaling["high_freq_factor"])
    long_wave, short_wave = orig / low, orig / high
    for i, f in enumerate(freqs):
        wave = 2.0 * math.pi / f
        if wave < short_wave:
            continue
        if wave > long_wave:
            freqs[i] = f / factor
        else:
            blend = (orig / wave - low) / (high - low)
            freqs[i] = (1.0 - blend) * f / factor + blend * f
    return freqs


def rope_magnitude(scaling: Optional[dict]) -> float:
    """The factor on cos and sin: 0.1 ln(factor) + 1 with scaling of type `yarn`, else 1."""
    if scaling and scaling.get("rope_type", scaling.get("type")) == "yarn":
        return 0.1 * math.log(float(scaling["factor"])) + 1.0
    return 1.0


@register_position("rope")
class RotaryEncoding(PositionEncoding):
    """params: head_dim, rotary_dim, theta, scaling (dict or None), layout ("half": channel i turns with
    channel i + rotary_dim/2, the default; "interleaved": channel 2i with channel 2i+1)."""

    def __init__(self, params):
        super().__init__(params)
        self.head_dim = int(params["head_dim"])
        self.rotary_dim = int(params.get("rotary_dim") or self.head_dim)
        self.theta = float(params["theta"])
        self.scaling = dict(params["scaling"]) if params.get("scaling") else None
        self.layout = str(params.get("layout", "half"))
        if self.layout not in ("half", "interleaved"):
            raise ValueError(f"rotary layout {self.layout!r}: known are 'half' and 'interleaved'")
        if self.rotary_dim % 2 or not 0 < self.rotary_dim <= self.head_dim:
            raise ValueError(f"rotary_dim {self.rotary_dim} must be even and at most head_dim {self.head_dim}")
        self.cos: Optional[torch.Tensor] = None
        self.sin: Optional[torch.Tensor] = None

    def tables(self, positions: int):
        """(cos, sin) as float64 CPU tensors [positions, rotary_dim/2]."""
        f = torch.tensor(rope_inv_freq(self.rotary_dim, self.theta, self.scaling), dtype=torch.float64)
        ang = torch.arange(positions, dtype=torch.float64)[:, None] * f[None, :]
        m = rope_magnitude(self.scaling)
        return torch.cos(ang) * m, torch.sin(ang) * m

    def prepare(self, ctx: BuildContext) -> None:
        super().prepare(ctx)
        c, s = self.tables(ctx.max_model_len)
        self.cos = c.to(torch.float32).to(ctx.device).contiguous()
        self.sin = s.to(torch.float32).to(ctx.device).contiguous()


@register_position("query_temperature")
class QueryTemperature(PositionEncoding):
    """A factor on the queries by position, 1 + coef * ln(floor((p + 1) / every) + 1).  params: coef, every.  `factor` is
    fp32 [positions], formed in float64."""

    def __init__(self, params):
        super().__init__(params)
        self.coef, self.every = float(params["coef"]), float(params["every"])
        if not self.every > 0:
            raise ValueError("query_temperature: `every` is positive")
        self.factor: Optional[torch.Tensor] = None

    def table(self, positions: int) -> torch.Tensor:
        p = torch.arange(positions, dtype=torch.float64)
        return 1.0 + self.coef * torch.log(torch.floor((p + 1.0) / self.every) + 1.0)

    def prepare(self, ctx: BuildContext) -> None:
        super().prepare(ctx)
        self.factor = self.table(ctx.max_model_len).to(torch.float32).to(ctx.device).contiguous()
