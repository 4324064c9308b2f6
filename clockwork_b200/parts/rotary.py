"""Rotate-half (neox) rotary position encoding, fused with the write of K and V into the cache.

Reference: ``clockwork/engine/model.py:171-175`` (``inv_freq[j] = 1 / theta^(2j/rotary_dim)`` in
float32), ``:186-191`` (angle = float(position) * inv_freq), ``:32-35`` and ``:92-95`` (element j
pairs with j + rotary_dim/2).  Parameters: ``theta``, ``rotary_dim``.  No tensors: ``inv_freq``
is derived (the reference keeps it out of checkpoints too, ``model.py:169``) and always float32.

``NoPosition`` stores K and V unrotated: the interface another position encoding must have is
``apply_and_store(ctx, qkv, view, num_heads, num_kv_heads, head_dim)``.

``rotary_tables`` is what mixers that rotate inside their own kernels make their frequencies with.
"""

from __future__ import annotations

import math

import torch

from .. import ops
from .base import PagedView, PositionEncoding, StepContext
from .registry import register_position


PAIRINGS = ("half", "interleaved")  # entry i with entry i + dims/2, or entry 2i with entry 2i + 1


def check_rotary(rotary: dict, dim: int) -> tuple:
    """(dims, base, interleaved) of a rotation ``{"dims", "base", "pairing", "scaling"}`` of heads of ``dim`` entries;
    ``pairing`` is "half" by default, ``scaling`` (absent or None: none) as ``rotary_tables`` takes it."""
    dims, base, pairing = int(rotary["dims"]), float(rotary["base"]), str(rotary.get("pairing", "half"))
    if dims <= 0 or dims % 2 or dims > dim or base <= 0:
        raise ValueError(f"rotary dims {dims} must be even, positive and at most dim {dim}, the base positive")
    if pairing not in PAIRINGS:
        raise ValueError(f"rotary pairing must be one of {PAIRINGS}, got {pairing!r}")
    scaling = rotary.get("scaling")
    if scaling is not None and (base == 1.0 or min(float(scaling[k]) for k in ("factor", "original", "fast", "slow")) <= 0):
        raise ValueError("a scaled rotation needs a base other than 1 and positive factor, original, fast and slow")
    return dims, base, pairing == "interleaved"


def rotary_tables(dims: int, base: float, scaling: dict | None = None) -> tuple[torch.Tensor, float]:
    """(angle per position of every pair, float32 [dims/2]; what sines and cosines are multiplied by).  Worked out in
    float64 and rounded once.  Plain: ``f_i = base^(-2i/dims)`` and 1.  With ``scaling`` = ``{"factor", "original", "fast",
    "slow"}`` (YaRN): pairs that turn more than ``fast`` times over ``original`` positions keep their frequency, pairs that
    turn less than ``slow`` times have it divided by ``factor``, a linear ramp over the pair's index between (its ends
    rounded outwards to whole indices); sines and cosines are multiplied by ``1 + 0.1 ln(factor)``."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    freq = base ** (-2.0 * i / dims)
    if scaling is None:
        return freq.to(torch.float32), 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def index_of(turns: float) -> float:  # of the pair that turns this often over `original` positions
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index_of(float(scaling["fast"]))), 0)
    hi = min(math.ceil(index_of(float(scaling["slow"]))), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return (freq / factor * ramp + freq * (1.0 - ramp)).to(torch.float32), 0.1 * math.log(factor) + 1.0


class RotaryNeox(PositionEncoding):
    graph_safe = True
    graph_safe_portions = True

    def __init__(self, spec, prefix, dtype, device) -> None:
        super().__init__(spec, prefix, dtype, device)
        self.theta = float(spec["theta"])
        self.rotary_dim = int(spec["rotary_dim"])
        if self.rotary_dim <= 0 or self.rotary_dim % 2:
            raise ValueError(f"rotary_dim {self.rotary_dim} must be positive and even")
        # the reference's expression, evaluated in float32 on the host, then uploaded
        exponents = torch.arange(0, self.rotary_dim, 2, dtype=torch.float32) / self.rotary_dim
        self.inv_freq = (1.0 / (self.theta**exponents)).to(device)

    def apply_and_store(self, ctx: StepContext, qkv: torch.Tensor, view: PagedView | None,
                        num_heads: int, num_kv_heads: int, head_dim: int) -> None:
        if self.rotary_dim > head_dim:
            raise ValueError(f"rotary_dim {self.rotary_dim} exceeds head_dim {head_dim}")
        write = view is not None and view.write
        ops.rope_store(qkv, ctx.positions, view.slots if write else None, self.inv_freq,
                       view.k_cache if write else None, view.v_cache if write else None,
                       num_heads, num_kv_heads, head_dim, self.rotary_dim, ctx.status, write_cache=write)


    def fused_decode_args(self, head_dim: int):
        """(inv_freq, rotary_dim) for kernels that apply this encoding themselves, or None."""
        return (self.inv_freq, self.rotary_dim) if self.rotary_dim <= head_dim else None


class NoPosition(PositionEncoding):
    graph_safe = True
    graph_safe_portions = True

    def fused_decode_args(self, head_dim: int):
        return (None, 0)

    def apply_and_store(self, ctx, qkv, view, num_heads, num_kv_heads, head_dim) -> None:
        if view is not None and view.write:
            ops.rope_store(qkv, ctx.positions, view.slots, None, view.k_cache, view.v_cache,
                           num_heads, num_kv_heads, head_dim, 0, ctx.status, write_cache=True)


class SinusoidalAbsolute(PositionEncoding):
    """A vector per position added to the embedding rows: entry 2i is ``sin(t * base^(-2i/size))`` and entry
    2i+1 the cosine of the same angle (float32 angles).  Parameters: ``size`` (the model's width), ``base``.  The
    model calls ``add_to_embedding`` once per step, with the scale of the embedding rows."""

    graph_safe = True
    graph_safe_portions = True

    def __init__(self, spec, prefix, dtype, device) -> None:
        super().__init__(spec, prefix, dtype, device)
        self.size, self.base = int(spec["size"]), float(spec.get("base", 10000.0))
        exponents = torch.arange(0, self.size, 2, dtype=torch.float64) / self.size
        self.inv_freq = (self.base ** -exponents).to(torch.float32).to(device)

    def add_to_embedding(self, x: torch.Tensor, positions: torch.Tensor, scale: float) -> None:
        ops.scale_add_sinusoid(x, positions, self.inv_freq, scale)


register_position("sinusoidal_absolute", SinusoidalAbsolute, replace=True)
register_position("rope_neox", RotaryNeox, replace=True)
register_position("none", NoPosition, replace=True)
