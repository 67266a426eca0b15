"""Position encodings a mixer can be given."""
from __future__ import annotations

import math

import numpy as np
import torch

from .. import ops
from ..config.specs import PositionSpec
from .base import PositionEncoding, register_position


def rope_inverse_frequencies(rotary_dim: int, theta: float) -> np.ndarray:
    """inv[i] = 1 / float32(theta ** float32(2i / rotary_dim)); the exponent is a
    32-bit quotient, the power is taken in 64-bit and rounded to 32-bit
    (buildRopeInvFreq, model.go:1742-1750)."""
    half = rotary_dim // 2
    i = (np.arange(half, dtype=np.float32) * np.float32(2.0))
    e = i / np.float32(rotary_dim)
    base = np.power(np.float64(theta), e.astype(np.float64)).astype(np.float32)
    return (np.float32(1.0) / base).astype(np.float32)


def stretched_frequencies(rotary_dim: int, theta: float, factor: float, original: float, fast: float, slow: float):
    """(64-bit frequencies [rotary_dim / 2], factor on the tables) of a rotation stretched to longer contexts the YaRN way:
    pairs that turn more than ``fast`` times over ``original`` positions keep theta^(-2i/d), pairs that turn less than
    ``slow`` times turn ``factor`` times slower, a linear ramp over the pairs between; cosine and sine are multiplied by
    0.1 ln(factor) + 1."""
    half = rotary_dim // 2
    inv = np.float64(theta) ** (-2.0 * np.arange(half, dtype=np.float64) / rotary_dim)

    def pair_of(turns):          # the pair (a real number) that turns so often over the original length
        return rotary_dim * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(theta))
    lo = max(math.floor(pair_of(fast)), 0)
    hi = min(math.ceil(pair_of(slow)), rotary_dim - 1)
    ramp = np.clip((np.arange(half, dtype=np.float64) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return inv / factor * ramp + inv * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def banded_frequencies(rotary_dim: int, theta: float, factor: float, low: float, high: float, original: float) -> np.ndarray:
    """64-bit frequencies [rotary_dim / 2] of a rotation stretched to longer contexts band by band, as Llama 3.1 does: with
    n = how often a pair turns over ``original`` positions, pairs with n > high keep theta^(-2i/d), pairs with n < low
    turn ``factor`` times slower, those between are blended linearly in n."""
    inv = np.float64(theta) ** (-2.0 * np.arange(rotary_dim // 2, dtype=np.float64) / rotary_dim)
    turns = original * inv / (2.0 * math.pi)
    share = np.clip((turns - low) / (high - low), 0.0, 1.0) if high > low else (turns >= low).astype(np.float64)
    return (1.0 - share) * inv / factor + share * inv


class Rope(PositionEncoding):
    """Rotary embedding over the first ``rotary_dim`` dims of a head.  The
    angle float32(pos) * inv[i] is a 32-bit product; sine and cosine are taken
    in 64-bit (prepareRopeScratch, model.go:3041-3046).  The tables depend on
    the step's positions only, so every layer of a step shares them.  Option ``exact_angles``: frequencies and angles
    in 64-bit; with it option ``yarn`` = (factor, original, fast, slow): see stretched_frequencies, or option ``bands`` =
    (factor, low, high, original): see banded_frequencies."""
    capturable = True
    launches_only = True

    def __init__(self, spec: PositionSpec):
        if spec.rotary_dim % 2:
            raise ValueError(f"rotary dimension {spec.rotary_dim} must be even")
        self.spec = spec
        self._inv = None
        self._gain = 1.0
        stretched = [k for k in ("yarn", "bands") if spec.option(k) is not None]
        if stretched and not spec.option("exact_angles", False):
            raise ValueError("stretched frequencies come with exact angles")
        if len(stretched) > 1:
            raise ValueError("frequencies are stretched one way or the other, not both")

    def tables(self, ctx):
        exact = bool(self.spec.option("exact_angles", False))
        yarn, bands = self.spec.option("yarn"), self.spec.option("bands")
        key = ("rope", self.spec.rotary_dim, float(self.spec.theta), exact, yarn, bands)
        hit = ctx.scratch.get(key)
        if hit is None:
            if self._inv is None or self._inv.device != ctx.device:
                if yarn is not None:
                    inv, self._gain = stretched_frequencies(self.spec.rotary_dim, float(self.spec.theta), *yarn)
                elif bands is not None:
                    inv = banded_frequencies(self.spec.rotary_dim, float(self.spec.theta), *bands)
                elif exact:
                    # frequencies theta^(-2i/d) and the angles pos * frequency in 64-bit: a table entry is then
                    # the rounded cosine of the true angle at any position (a 32-bit angle is off by up to
                    # position * 2^-24 radians, which a sharp head sees a thousand positions on)
                    half = self.spec.rotary_dim // 2
                    inv = np.float64(self.spec.theta) ** (-2.0 * np.arange(half, dtype=np.float64) / self.spec.rotary_dim)
                else:
                    inv = rope_inverse_frequencies(self.spec.rotary_dim, self.spec.theta)
                self._inv = torch.from_numpy(inv).to(ctx.device)
            hit = ops.rope_table(ctx.tok_pos, self._inv, self._gain)
            ctx.scratch[key] = hit
        return hit


class NoPosition(PositionEncoding):
    capturable = True
    launches_only = True
    def __init__(self, spec: PositionSpec):
        self.spec = spec

    def tables(self, ctx):
        return None


register_position("rope", Rope)
register_position("none", NoPosition)
