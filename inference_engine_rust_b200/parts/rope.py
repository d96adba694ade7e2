"""Rotary position encoding as a part: its constants (theta, how many dimensions rotate,
which elements pair up) are parameters; a mixer's kernel may apply the rotation itself
(`rotary_constants`: fused with its cache write, or with its attention in one-token steps).

angle(pos, k) = pos * theta^(-2k / rotary_dim), computed in fp32 on the device from a
table of theta^(-2k / rotary_dim) made here in double precision.  (The reference reaches
the same angle by repeated fp32 multiplication, src/ops/rope.rs:40-57; the two differ by
that loop's rounding only.)  `yarn` (factor, original, fast, slow) stretches the rotation for
contexts longer than `original`: pairs that turn at least `fast` times within `original` positions keep
their rate, pairs that turn at most `slow` times are slowed down by `factor`, the rates between are
mixed linearly in the pair's number, and cosine and sine are multiplied by 0.1 ln(factor) + 1 (the YaRN
method of Peng, Quesnelle, Fan and Shippole, "YaRN: Efficient Context Window Extension of Large Language
Models").  Pairing "interleaved" rotates (2k, 2k+1) as the reference
does on its row-permuted tensors; "half" rotates (k, k + rotary_dim/2), which is the same
rotation on tensors in safetensors row order (src/layers/attention.rs:137-172).
"""
from __future__ import annotations

import math

import torch

from ..csrc import bindings as B
from .base import PositionEncoding, Runtime, register_part

PAIRINGS = {"half": B.PAIR_HALF, "interleaved": B.PAIR_INTERLEAVED}


def yarn_rates(theta: float, rotary_dim: int, factor: float, original: float, fast: float, slow: float):
    """(radians per position of every pair, in double precision; the factor on cosine and sine)."""
    k = torch.arange(rotary_dim // 2, dtype=torch.float64)
    plain = torch.pow(torch.tensor(theta, dtype=torch.float64), -2.0 * k / max(rotary_dim, 1))

    def pair_that_turns(times: float) -> float:
        return rotary_dim * math.log(original / (2.0 * math.pi * times)) / (2.0 * math.log(theta))
    lo = max(math.floor(pair_that_turns(fast)), 0)
    hi = min(math.ceil(pair_that_turns(slow)), rotary_dim - 1)
    slowed = torch.clamp((k - lo) / max(hi - lo, 0.001), 0.0, 1.0)      # 0: as it is, 1: divided by the factor
    return plain / factor * slowed + plain * (1.0 - slowed), 0.1 * math.log(factor) + 1.0


class RotaryEncoding(PositionEncoding):
    def __init__(self, spec, head_dim: int, rt: Runtime):
        self.theta = float(spec["theta"])
        self.head_dim = head_dim
        self.rotary_dim = int(spec.get("rotary_dim", head_dim))
        pairing = spec.get("pairing", "half")
        if pairing not in PAIRINGS:
            raise ValueError(f"rope pairing must be one of {sorted(PAIRINGS)}, got {pairing!r}")
        if self.rotary_dim % 2 or not 0 <= self.rotary_dim <= head_dim:
            raise ValueError(f"rotary_dim {self.rotary_dim} must be even and at most head_dim {head_dim}")
        self.pairing = PAIRINGS[pairing]
        k = torch.arange(self.rotary_dim // 2, dtype=torch.float64)
        inv = torch.pow(torch.tensor(self.theta, dtype=torch.float64), -2.0 * k / max(self.rotary_dim, 1))
        factors = spec.get("freq_factors")       # optional per-pair divisors (src/ops/rope.rs:45-50)
        if factors is not None:
            inv = inv / torch.as_tensor(factors, dtype=torch.float64)
        self.multiplier = 1.0                    # on cosine and sine
        yarn = spec.get("yarn")
        if yarn is not None:
            if factors is not None:
                raise ValueError("rope takes freq_factors or yarn, not both")
            inv, self.multiplier = yarn_rates(self.theta, self.rotary_dim, float(yarn["factor"]), float(yarn["original"]),
                                              float(yarn["fast"]), float(yarn["slow"]))
        self.inv_freq = inv.to(torch.float32).to(rt.device)

    def rotary_constants(self):
        return (self.inv_freq, self.rotary_dim, self.pairing) if self.multiplier == 1.0 else None

    def scaled_rotary_constants(self):
        return self.inv_freq, self.rotary_dim, self.pairing, self.multiplier

    def encode(self, qkv, ctx, heads: int, kv_heads: int) -> None:
        B.rotate_qk(qkv, ctx.batch, self.inv_freq, heads, kv_heads, self.head_dim, self.rotary_dim, self.pairing,
                    ctx.rt.err, ctx.stream, rot_mul=self.multiplier)


register_part("position", "rope", RotaryEncoding)
