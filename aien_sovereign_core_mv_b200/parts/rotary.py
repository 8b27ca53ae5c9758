"""Rotary position encoding: frequency table, optional llama3 smoothing or YaRN ramp, per-step cos/sin."""
from __future__ import annotations

import math
from typing import Optional

import torch

from .. import kernels as K
from ..registry import register_position
from .base import Position, StepContext


def inverse_frequencies(head_dim: int, theta: float, scaling: Optional[dict] = None, rotary_dim: Optional[int] = None,
                        theta_as_float32: bool = True, linear_factor: float = 1.0):
    """inv_freq_i = theta^(-2i/d) in float64 (theta itself held as float32, as the reference
    does, unless ``theta_as_float32`` is off), optionally smoothed the llama3 way
    (crates/aien-abi-core/src/lib.rs:69-84, 106-114)."""
    d = rotary_dim or head_dim
    theta32 = float(torch.tensor(theta, dtype=torch.float32).item()) if theta_as_float32 else float(theta)
    inv = [1.0 / theta32 ** ((2 * i) / d) for i in range(d // 2)]
    if scaling:
        old = float(scaling["original_max_position_embeddings"])
        low_w = old / scaling["low_freq_factor"]
        high_w = old / scaling["high_freq_factor"]
        out = []
        for f in inv:
            wavelen = 2.0 * math.pi / f
            if wavelen < high_w:
                out.append(f)
            elif wavelen > low_w:
                out.append(f / scaling["factor"])
            else:
                smooth = (old / wavelen - scaling["low_freq_factor"]) / (scaling["high_freq_factor"] - scaling["low_freq_factor"])
                out.append((1.0 - smooth) * f / scaling["factor"] + smooth * f)
        inv = out
    if linear_factor and float(linear_factor) != 1.0:
        inv = [f / float(linear_factor) for f in inv]          # linear scaling: every frequency divided by one factor
    return inv


def yarn_frequencies(dims: int, theta: float, factor: float, original: float, fast: float, slow: float):
    """(frequencies, factor on cos and sin).  A pair that turns often within ``original`` positions keeps its frequency, one
    that turns seldom takes it divided by ``factor``; between the pair indices that turn ``fast`` and ``slow`` times the two
    are mixed linearly in the index.  Both tables are multiplied by 0.1 ln(factor) + 1."""
    def pair_that_turns(times):
        return dims * math.log(original / (2.0 * math.pi * times)) / (2.0 * math.log(theta))

    lo, hi = max(math.floor(pair_that_turns(fast)), 0), min(math.ceil(pair_that_turns(slow)), dims - 1)
    span = max(hi - lo, 0.001)
    out = []
    for i in range(dims // 2):
        f, r = theta ** (-2.0 * i / dims), min(max((i - lo) / span, 0.0), 1.0)
        out.append(f / factor * r + f * (1.0 - r))
    return out, 0.1 * math.log(factor) + 1.0


@register_position("rotary")
class RotaryPosition(Position):
    """angle = position * inv_freq in float64, cos and sin rounded to float32
    (crates/aien-inference-abi/src/tensor.rs:150-188).  The table of a step is built once and
    shared by every layer that uses the same part.  ``pairing`` says which dimensions a mixer
    rotates together: "halves" (i with i + d/2, rotate_half) or "interleaved" (2i with 2i+1); the
    table is the same, the mixer's kernel reads ``pairing``.  ``linear_factor`` f: every frequency is divided by f.
    ``yarn`` {factor, original, fast, slow}: see :func:`yarn_frequencies`."""

    def __init__(self, head_dim: int, theta: float, scaling: Optional[dict] = None, rotary_dim: Optional[int] = None,
                 pairing: str = "halves", theta_as_float32: bool = True, linear_factor: float = 1.0,
                 yarn: Optional[dict] = None):
        if pairing not in ("halves", "interleaved"):
            raise ValueError(f"rotary pairing {pairing!r}: 'halves' or 'interleaved'")
        self.pairing = pairing
        self.head_dim = int(head_dim)
        self.rotary_dim = int(rotary_dim or head_dim)
        if self.rotary_dim % 2 or self.rotary_dim > self.head_dim:
            raise ValueError(f"rotary_dim {self.rotary_dim} must be even and at most head_dim {self.head_dim}")
        self.theta = float(theta)
        self.scaling = dict(scaling) if scaling else None
        self.linear_factor = float(linear_factor or 1.0)
        if self.linear_factor <= 0.0:
            raise ValueError(f"linear_factor {linear_factor!r} must be positive")
        if yarn and (scaling or self.linear_factor != 1.0):
            raise ValueError("one frequency scaling at a time")
        self.mult = 1.0
        self._inv_host = inverse_frequencies(self.head_dim, self.theta, self.scaling, self.rotary_dim, bool(theta_as_float32), self.linear_factor)
        if yarn:
            self._inv_host, self.mult = yarn_frequencies(self.rotary_dim, self.theta, float(yarn["factor"]), float(yarn["original"]),
                                                         float(yarn["fast"]), float(yarn["slow"]))
        self._inv_dev: Optional[torch.Tensor] = None

    def step_workspace_bytes(self, max_tokens):
        return 2 * (max_tokens * (self.rotary_dim // 2) * 4 + 256)

    def rotary(self, ctx: StepContext):
        key = ("rotary", id(self))
        hit = ctx.shared.get(key)
        if hit is None:
            if self._inv_dev is None:
                self._inv_dev = torch.tensor(self._inv_host, dtype=torch.float64, device=ctx.positions.device)
            half = self.rotary_dim // 2
            cos = ctx.workspace.take_step((ctx.num_tokens, half), torch.float32)
            sin = ctx.workspace.take_step((ctx.num_tokens, half), torch.float32)
            K.rope_table(ctx.positions, self._inv_dev, cos, sin, self.mult)
            hit = (cos, sin, self.rotary_dim)
            ctx.shared[key] = hit
        return hit


@register_position("none")
class NoPosition(Position):
    """Positions enter nowhere (a mixer with its own notion of order)."""

    def __init__(self, **_):
        pass

    def rotary(self, ctx):
        return None

    def apply(self, ctx, q, group, run):
        return None
