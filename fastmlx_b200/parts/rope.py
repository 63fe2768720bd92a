"""Rotary position encoding, fused with the write of k and v into the layer's pages."""
from __future__ import annotations

import math

import torch

from ..config.llama import YarnScaling
from .base import PositionEncoding, Runtime


def inverse_frequencies(rotary_dim: int, theta: float, scaling=None) -> torch.Tensor:
    """f_j = theta^(-2j/dims), j < dims/2, in float64 (tamnd/fastmlx passes base=rope_theta,
    dims=head_dim, scale=1 to the fused rope: compute/models/llama.go:377,411-412,
    compute/models/qwen3_forward.go:153-172).

    `scaling` (a config.llama.RopeScaling of type llama3; the reference parses the block,
    compute/testdata/llama_args.json:161-183, and never applies it) rescales by wavelength
    l_j = 2 pi / f_j: shorter than orig/high_freq_factor keeps f_j; longer than
    orig/low_freq_factor gives f_j/factor; between, with s = (orig/l_j - low)/(high - low),
    (1 - s) f_j/factor + s f_j.  A `YarnScaling` blends by pair number instead: pair i keeps f_i up to lo and gets
    f_i/factor from hi on, linear in between, lo and hi being the pairs that turn `fast` and `slow` times over the original
    length, t(n) = dims ln(original / (2 pi n)) / (2 ln theta), rounded down and up and clipped to [0, dims - 1]."""
    j = torch.arange(0, rotary_dim, 2, dtype=torch.float64)
    f = torch.pow(torch.tensor(float(theta), dtype=torch.float64), -j / rotary_dim)
    if scaling is None:
        return f
    if isinstance(scaling, YarnScaling):
        def pair_of(turns):
            return rotary_dim * math.log(scaling.original / (2 * math.pi * turns)) / (2 * math.log(theta))
        lo, hi = max(math.floor(pair_of(scaling.fast)), 0), min(math.ceil(pair_of(scaling.slow)), rotary_dim - 1)
        ramp = ((j / 2 - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        return f / scaling.factor * ramp + f * (1.0 - ramp)
    orig = float(scaling.original_max_position_embeddings)
    lo, hi, factor = scaling.low_freq_factor, scaling.high_freq_factor, scaling.factor
    lam = 2 * math.pi / f
    s = (orig / lam - lo) / (hi - lo)
    mid = (1 - s) * f / factor + s * f
    return torch.where(lam < orig / hi, f, torch.where(lam > orig / lo, f / factor, mid))


class RotaryEmbedding(PositionEncoding):
    """Rotates pairs of q and k by position * f_j (angle, sine and cosine in 32-bit).
    `traditional` pairs (2j, 2j+1), otherwise (j, j + rotary_dim/2).  It has no tensors in
    the checkpoint; the table is built once, in float64, and held in 32-bit."""

    def __init__(self, head_dim: int, theta: float, scaling=None, traditional: bool = False,
                 rotary_dim: int | None = None):
        self.head_dim = int(head_dim)
        self.rotary_dim = int(rotary_dim if rotary_dim is not None else head_dim)
        if self.rotary_dim % 2 or not 0 <= self.rotary_dim <= self.head_dim:
            raise ValueError(f"rotary_dim {self.rotary_dim} must be even and at most head_dim {self.head_dim}")
        self.theta, self.scaling, self.traditional = float(theta), scaling, bool(traditional)
        self.amplitude = float(getattr(scaling, "amplitude", 1.0))
        self.inv_freq = None

    def bind_own(self, tensors, rt: Runtime):
        self.inv_freq = inverse_frequencies(self.rotary_dim, self.theta, self.scaling) \
            .to(torch.float32).to(rt.device).contiguous()

    def apply_and_store(self, qkv, ctx, cache, nh, nkv, hd):
        if self.amplitude != 1.0:
            raise ValueError("a rotation with an amplitude runs on the route with 32-bit scores (qk_prepare)")
        g = ctx.groups[cache.group] if cache.kv is not None else None
        self.rt.k.rope_kv_write(
            qkv, ctx.positions, self.inv_freq, self.rotary_dim, self.traditional,
            g.slot_mapping if (g is not None and cache.writable) else None,
            cache.kv if cache.writable else None,
            nh, nkv, hd, ctx.status)


    def fused_args(self, cache):
        """What a mixer kernel needs to rotate and store by itself: (frequencies, rotated
        width, pairing, whether to store k and v)."""
        return (self.inv_freq, self.rotary_dim, self.traditional, bool(cache.kv is not None and cache.writable))

    def native_args(self):
        return (self.inv_freq, self.rotary_dim, self.traditional)


class NoPositionEncoding(PositionEncoding):
    """Stores k and v unrotated (a mixer whose positions come from elsewhere)."""

    def apply_and_store(self, qkv, ctx, cache, nh, nkv, hd):
        g = ctx.groups[cache.group] if cache.kv is not None else None
        self.rt.k.rope_kv_write(
            qkv, ctx.positions, None, 0, False,
            g.slot_mapping if (g is not None and cache.writable) else None,
            cache.kv if cache.writable else None,
            nh, nkv, hd, ctx.status)

    def fused_args(self, cache):
        return (None, 0, False, bool(cache.kv is not None and cache.writable))

    def native_args(self):
        return (None, 0, False)
