"""A matrix memory with exponential gates (the matrix form of an extended LSTM), as a mixer."""
from __future__ import annotations

import torch

from .base import Mixer, Runtime, StateSpec, WeightSpec, to_f32_vector
from .linear import Linear


class MatrixMemoryMixer(Mixer):
    """q = W_q x * dim^-1/2 and k = W_k x (heads x dim), v = W_v x (heads x vdim).  Per head a log input gate
    i = cap tanh((W_i x + b_i) / cap) and a log forget gate f = logsigmoid(cap tanh((W_f x + b_f) / cap)).  With S [dim, vdim],
    n [dim] and a running maximum m, all starting at zero and carried from token to token in 32-bit,

        m' = max(f + m, i);   S <- exp(f + m - m') S + exp(i - m') k v^T;   n likewise with k alone;   m <- m'
        o = S^T q / (max(|n . q|, exp(-m)) + 1e-6)

    Each head's o is divided by its root mean square (eps `norm_eps`); the heads side by side are multiplied by a weight of
    their whole width and by sigmoid(W_g x), and go through the output projection.

    Per request the part keeps, in one state slot of 32-bit floats, S^T of every head with n as one more row
    ([heads, vdim + 1, dim]) and m of every head.  Everything between the projections and the gated read-out is 32-bit, and so
    is the gates' projection.  Steps of single tokens run gates, recurrence, norm and output gate in one kernel; steps with
    portions work the gates out over each row's tokens first, walk the recurrence from them, and divide, norm and gate after it.
    `names`: the tensors of (q, k, v, g, i, f, o, norm); the gates' biases are `<i><bias_suffix>`, `<f><bias_suffix>`.
    `output=False` leaves the output projection to the block."""

    supports_cuda_graph = True
    WIDE_MAX_TOKENS = 16          # up to so many tokens all projections are one product that leaves in 32-bit

    def __init__(self, width: int, heads: int, dim: int, vdim: int, gate_cap: float, norm_eps: float, name: str,
                 names=("q", "k", "v", "g", "i", "f", "o", "norm"), output: bool = True, weight_suffix: str = ".weight",
                 bias_suffix: str = ".b"):
        if dim > 512:
            raise ValueError(f"the recurrence keeps up to 512 rows of state per column, not {dim}")
        if not gate_cap > 0:
            raise ValueError(f"the gates' cap must be positive, not {gate_cap}")
        self.H, self.D, self.Dv, self.cap, self.eps = int(heads), int(dim), int(vdim), float(gate_cap), float(norm_eps)
        q, k, v, g, i, f, o, norm = (f"{name}.{n}" for n in names)
        self.inner_features = self.H * self.Dv
        # rows: q | k | v | output gate | input gates | forget gates
        self.proj = Linear(width, [(q, self.H * self.D), (k, self.H * self.D), (v, self.inner_features), (g, self.inner_features),
                                   (i, self.H), (f, self.H)], weight_suffix=weight_suffix)
        self.bias_names, self.norm_name = (i + bias_suffix, f + bias_suffix), norm
        self.out_piece = (o + weight_suffix, self.inner_features, None)
        self.o = Linear(self.inner_features, [(o, width)], weight_suffix=weight_suffix) if output else None
        self.s_floats = self.H * (self.Dv + 1) * self.D

    def children(self):
        return tuple(p for p in (self.proj, self.o) if p is not None)

    def own_weight_specs(self):
        return [WeightSpec(self.bias_names[0], (self.H,), "bias"), WeightSpec(self.bias_names[1], (self.H,), "forget_bias"),
                WeightSpec(self.norm_name, (self.inner_features,), "norm")]

    def bind_own(self, tensors, rt: Runtime):
        self.gate_bias = torch.cat([to_f32_vector(tensors[n], rt) for n in self.bias_names]).contiguous()
        self.norm_w = to_f32_vector(tensors[self.norm_name], rt)

    def weight_bytes(self):
        return super().weight_bytes() + 4 * (2 * self.H + self.inner_features)

    def state_spec(self):
        # a multiple of four floats, so that every slot starts on 16 bytes
        return StateSpec((-(-(self.s_floats + self.H) // 4) * 4,), torch.float32)

    def forward_inner(self, x, ctx, cache, out=None):
        """The normalised, gated read-outs of all heads side by side, [T, heads * vdim]."""
        k, w = self.rt.k, self.proj.weight
        n, m = 2 * self.H * self.D + self.inner_features, self.inner_features
        if x.shape[0] <= self.WIDE_MAX_TOKENS:
            proj = k.linear(x, w, None, torch.float32)
            z = proj[:, n + m:]
        else:
            proj = k.linear(x, w[:n + m], None, self.rt.dtype)
            z = k.linear(x, w[n + m:], None, torch.float32)
        if ctx.max_q_len == 1:
            return k.mlstm_step(proj, z, self.gate_bias, self.cap, ctx, cache.state, self.H, self.D, self.Dv, self.norm_w, self.eps,
                                self.rt.dtype, out=out)
        gates = k.mlstm_gates(z, self.gate_bias, self.cap, ctx, cache.state, self.s_floats, self.H)
        o, nq = k.mlstm_scan(proj, gates, ctx, cache.state, self.H, self.D, self.Dv)
        return k.head_norm_gate(o, proj[:, n:n + m], self.norm_w, self.eps, self.H, self.Dv, self.rt.dtype, "sigmoid", out=out,
                                divisor=(nq, gates))

    def forward(self, x, ctx, cache):
        return self.o.forward(self.forward_inner(x, ctx, cache))
