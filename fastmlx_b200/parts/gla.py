"""Gated linear attention: a matrix of state per head whose rows decay each by a factor of the token's own."""
from __future__ import annotations

import torch

from .base import FreeDim, Mixer, Runtime, StateSpec, WeightSpec, to_f32_vector
from .linear import BlockDiagonalLinear, Linear


class GatedLinearAttention(Mixer):
    """q = W_q x * dim^-1/2 and k = W_k x (heads x dim), v = W_v x (heads x vdim); a decay per head and key channel, alpha =
    sigmoid(W_a2 (W_a1 x) + bias)^(1/tau).  Per head, with S [dim, vdim] carried from token to token in 32-bit and starting
    at zero,

        S <- diag(alpha) S + k v^T;   o = S^T q

    with neither a softmax nor a denominator.  Each head's o is divided by its root mean square (eps `norm_eps`), multiplied by
    a weight shared by the heads; the heads side by side are multiplied by silu(W_g x) and go through the output projection.

    The rank of the decays' projection is read from the checkpoint (`rank` is its size in random weights).  Per request
    the part keeps S^T of every head ([heads, vdim, dim]) in one state slot of 32-bit floats.  Everything between the
    projections and the gated read-out is 32-bit.  `names`: the tensors of (q, k, v, g, a1, a2, o, norm); the decays' bias
    is `<a2><bias_suffix>`.  `output=False` leaves the output projection to the block."""

    supports_cuda_graph = True

    def __init__(self, width: int, heads: int, dim: int, vdim: int, tau: float, norm_eps: float, name: str,
                 names=("q", "k", "v", "g", "a1", "a2", "o", "norm"), output: bool = True, weight_suffix: str = ".weight",
                 bias_suffix: str = ".b", rank: int | None = None):
        if dim > 512:
            raise ValueError(f"the recurrence keeps up to 512 rows of state per column, not {dim}")
        if not tau > 0:
            raise ValueError(f"the decays' root must be positive, not {tau}")
        self.H, self.D, self.Dv, self.tau, self.eps = int(heads), int(dim), int(vdim), float(tau), float(norm_eps)
        q, k, v, g, a1, a2, o, norm = (f"{name}.{n}" for n in names)
        self.inner_features = self.H * self.Dv
        ra = FreeDim(int(rank) if rank else 16, a1)
        # one product: q | k | v | gate | first half of the decays' projection
        self.proj = Linear(width, [(q, self.H * self.D), (k, self.H * self.D), (v, self.inner_features), (g, self.inner_features), (a1, ra)],
                           weight_suffix=weight_suffix)
        self.second = BlockDiagonalLinear([(a2 + weight_suffix, self.H * self.D, ra)])
        self.bias_name, self.norm_name = a2 + bias_suffix, norm
        self.out_piece = (o + weight_suffix, self.inner_features, None)
        self.o = Linear(self.inner_features, [(o, width)], weight_suffix=weight_suffix) if output else None
        self.s_floats = self.H * self.Dv * self.D
        self.out_scale = 1.0

    def children(self):
        return tuple(p for p in (self.proj, self.second, self.o) if p is not None)

    def own_weight_specs(self):
        return [WeightSpec(self.bias_name, (self.H * self.D,), "bias"), WeightSpec(self.norm_name, (self.Dv,), "norm")]

    def bind_own(self, tensors, rt: Runtime):
        self.bias, self.norm_w = (to_f32_vector(tensors[n], rt) for n in (self.bias_name, self.norm_name))
        if self.out_scale != 1.0:
            self.norm_w = (self.norm_w * self.out_scale).contiguous()

    def scale_output(self, s: float) -> None:
        """What `forward_inner` hands on is multiplied by s (it rides in the norm's 32-bit weight)."""
        self.out_scale = float(s)

    def weight_bytes(self):
        return super().weight_bytes() + 4 * (self.H * self.D + self.Dv)

    def state_spec(self):
        # a multiple of four floats, so that every slot starts on 16 bytes
        return StateSpec((-(-self.s_floats // 4) * 4,), torch.float32)

    def forward_inner(self, x, ctx, cache, out=None, proj=None):
        """The normalised, gated read-outs of all heads side by side, [T, heads * vdim]."""
        k = self.rt.k
        if proj is None:
            proj = self.proj.forward(x)
        n, m = 2 * self.H * self.D + self.inner_features, self.inner_features
        z = self.second.forward(proj[:, n + m:n + m + self.second.in_features], out_dtype=torch.float32)
        qkv, alpha = k.channel_gla_prepare(proj, z, self.bias, self.H, self.D, self.Dv, self.D ** -0.5, self.tau)
        o = k.channel_scan(qkv, alpha, None, ctx, cache.state, self.H, self.H, self.D, self.Dv)
        return k.head_norm_gate(o, proj[:, n:n + m], self.norm_w, self.eps, self.H, self.Dv, self.rt.dtype, "silu", out=out)

    def forward(self, x, ctx, cache):
        return self.o.forward(self.forward_inner(x, ctx, cache))
