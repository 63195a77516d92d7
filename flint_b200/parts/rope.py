"""Rotary position encoding with optional linear, banded, LongRoPE or YaRN scaling.

The cos/sin tables are built on the host in float64 and stored as float32
[positions, rotary_dim/2]: inv_i = theta^(-2i/rot), divided by the short factor for
positions below the original context length and by the long factor from there on.
The choice is made per position, as the reference does
(crates/thuban_model/src/ops/rope.rs:52-87), so a cached key never has to be rotated
again and the logits do not depend on how a prompt was cut.  The LongRoPE magnitude
scale (short_mscale / long_mscale, again per position) multiplies cos and sin; the
reference has no such scale.  The rotation itself (dims i and i + rot/2 together, or, with
style "interleaved", dims 2i and 2i + 1) is done by the kernel that also writes the cache.
"""
from __future__ import annotations

import math

import torch

from ..errors import ConfigError
from ..registry import POSITION_ENCODINGS
from .base import PositionEncoding


@POSITION_ENCODINGS.register("rope")
class RotaryEncoding(PositionEncoding):
    """params: rotary_dim, theta, max_positions, style ("half", the default, or "interleaved"), and for LongRoPE:
    short_factor, long_factor, original_max_positions, short_mscale, long_mscale.  For YaRN: ``yarn`` = {factor,
    original, fast, slow}: with dim(t) = rot ln(original / (2 pi t)) / (2 ln theta), lo = max(floor(dim(fast)), 0),
    hi = min(ceil(dim(slow)), rot - 1) and ramp_i = clamp((i - lo) / max(hi - lo, 0.001), 0, 1), frequency i is
    inv_i / factor * ramp_i + inv_i (1 - ramp_i), and cos and sin are multiplied by 0.1 ln(factor) + 1.  ``linear`` =
    factor: every frequency is divided by it.  ``banded`` = {factor, low, high, original} (as in Llama 3.1): with the
    wavelength l = 2 pi / inv_i, frequency i stays for l < original / high, is divided by the factor for l > original / low,
    and between the two is (1 - s) inv_i / factor + s inv_i with s = (original / l - low) / (high - low).  The tables
    cover the positions the model is built to serve (``BuildContext.max_context``) when that is fewer than
    ``max_positions``."""

    def __init__(self, params, ctx):
        super().__init__(params, ctx)
        self.rotary_dim = int(params["rotary_dim"])
        if self.rotary_dim <= 0 or self.rotary_dim % 2:
            raise ConfigError(f"rotary_dim must be even and positive, got {self.rotary_dim}")
        self.theta = float(params["theta"])
        self.max_positions = int(params["max_positions"])
        if getattr(ctx, "max_context", None):
            self.max_positions = min(self.max_positions, int(ctx.max_context))
        self.style = params.get("style", "half")
        if self.style not in ("half", "interleaved"):
            raise ConfigError(f"rotation style must be 'half' or 'interleaved', got {self.style!r}")
        self._tables = None

    def tables(self):
        if self._tables is None:
            half = self.rotary_dim // 2
            i = torch.arange(half, dtype=torch.float64)
            inv = self.theta ** (-2.0 * i / self.rotary_dim)
            pos = torch.arange(self.max_positions, dtype=torch.float64)
            p = self.params
            if p.get("short_factor") is not None:
                short = torch.tensor(p["short_factor"], dtype=torch.float64)
                long = torch.tensor(p["long_factor"], dtype=torch.float64)
                if short.numel() != half or long.numel() != half:
                    raise ConfigError(f"LongRoPE factor lists must have {half} entries")
                is_short = (pos < int(p["original_max_positions"]))[:, None]
                ang = pos[:, None] * torch.where(is_short, inv / short, inv / long)
                scale = torch.where(is_short, torch.tensor(float(p.get("short_mscale", 1.0)), dtype=torch.float64),
                                    torch.tensor(float(p.get("long_mscale", 1.0)), dtype=torch.float64))
            elif p.get("yarn") is not None:
                y = p["yarn"]
                factor, original = float(y["factor"]), float(y["original"])
                if factor <= 0 or original <= 0 or float(y["fast"]) <= 0 or float(y["slow"]) <= 0 or self.theta <= 1:
                    raise ConfigError("YaRN: factor, original, fast and slow must be positive (and theta above 1)")
                where = lambda t: self.rotary_dim * math.log(original / (2 * math.pi * t)) / (2 * math.log(self.theta))
                lo = max(math.floor(where(float(y["fast"]))), 0)
                hi = min(math.ceil(where(float(y["slow"]))), self.rotary_dim - 1)
                ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0, 1)
                ang = pos[:, None] * (inv / factor * ramp + inv * (1 - ramp))[None, :]
                scale = torch.full((1, 1), 0.1 * math.log(factor) + 1, dtype=torch.float64)
            elif p.get("banded") is not None:
                b = {k: float(p["banded"][k]) for k in ("factor", "low", "high", "original")}
                if min(b.values()) <= 0 or b["high"] < b["low"]:
                    raise ConfigError("banded frequencies: factor, low, high and original must be positive, high at least low")
                turns = b["original"] * inv / (2 * math.pi)           # original / wavelength
                share = ((turns - b["low"]) / max(b["high"] - b["low"], 1e-30)).clamp(0, 1)
                ang = pos[:, None] * torch.where(turns > b["high"], inv, torch.where(
                    turns < b["low"], inv / b["factor"], (1 - share) * inv / b["factor"] + share * inv))[None, :]
                scale = torch.ones((1, 1), dtype=torch.float64)
            else:
                if p.get("linear") is not None:
                    if float(p["linear"]) <= 0:
                        raise ConfigError(f"the frequencies' divisor must be positive, got {p['linear']}")
                    inv = inv / float(p["linear"])
                ang = pos[:, None] * inv[None, :]
                scale = torch.ones((1, 1), dtype=torch.float64)
            cos = (torch.cos(ang) * scale).to(torch.float32).contiguous().to(self.ctx.device)
            sin = (torch.sin(ang) * scale).to(torch.float32).contiguous().to(self.ctx.device)
            self._tables = (cos, sin)
        return self._tables
