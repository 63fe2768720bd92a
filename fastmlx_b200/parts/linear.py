"""y = x W^T (+ b), W stored [out, in]."""
from __future__ import annotations

import torch

from .base import FreeDim, Part, Runtime, WeightSpec, to_compute, to_f32_vector


class Linear(Part):
    """One or several checkpoint matrices applied as a single product: `names` lists
    (tensor name prefix, out features); their rows are stacked at bind time, so q/k/v or
    gate/up run as one matrix product (tamnd/fastmlx runs them one by one,
    compute/models/llama.go:403-405,426-427, through compute/models/qwen3_forward.go:111-115)."""

    def __init__(self, in_features: int, names, bias: bool = False, interleave: int = 0,
                 weight_suffix: str = ".weight", bias_suffix: str = ".bias"):
        """The suffixes complete a tensor's name (a checkpoint that calls its matrices `x.q` and their
        biases `x.q.b` passes "" and ".b").  `interleave` = b > 0 (two matrices of equal height, a multiple of b): their rows are
        stacked in alternating blocks of b, so that a tile of 2b output columns holds b rows
        of the first and the matching b rows of the second."""
        self.in_features = int(in_features)
        self.names = [(n, o if isinstance(o, FreeDim) else int(o)) for n, o in names]
        self.out_features = sum(o for _, o in self.names)         # (a `FreeDim`'s true size is known once bound)
        self.has_bias = bool(bias)
        self.interleave = int(interleave)
        self.wsfx, self.bsfx = weight_suffix, bias_suffix
        if self.interleave and (len(self.names) != 2 or self.names[0][1] != self.names[1][1]
                                or self.names[0][1] % self.interleave):
            raise ValueError("interleaving takes two matrices of equal height, a multiple of the block")
        self.weight = None
        self.bias = None

    def own_weight_specs(self):
        specs = [WeightSpec(n + self.wsfx, (o, self.in_features), "matrix") for n, o in self.names]
        if self.has_bias:
            specs += [WeightSpec(n + self.bsfx, (o,), "bias") for n, o in self.names]
        return specs

    def bind_own(self, tensors, rt: Runtime):
        ws = [to_compute(tensors[n + self.wsfx], rt) for n, _ in self.names]
        if len({w.dtype for w in ws}) > 1:
            ws = [w.float() for w in ws]
        bs = [to_f32_vector(tensors[n + self.bsfx], rt) for n, _ in self.names] if self.has_bias else None
        if self.interleave:
            b = self.interleave
            ws = [torch.stack([w.view(-1, b, self.in_features) for w in ws], dim=1).reshape(-1, self.in_features)]
            if bs is not None:
                bs = [torch.stack([v.view(-1, b) for v in bs], dim=1).reshape(-1)]
        self.weight = ws[0].contiguous() if len(ws) == 1 else torch.cat(ws, dim=0).contiguous()
        self.out_features = self.weight.shape[0]
        if bs is not None:
            self.bias = torch.cat(bs).contiguous()

    def weight_bytes(self):
        return self.weight.numel() * self.weight.element_size()

    def forward(self, x, out_dtype=None):
        return self.rt.k.linear(x, self.weight, self.bias, out_dtype or self.rt.dtype)

    def emit(self, b, x: int, out_dtype=None, out: int | None = None) -> int:
        """Native program: out = x . W^T (+ b) into a new register (or into `out`)."""
        from ..engine.native import OP_LINEAR, _dt
        dt = _dt(out_dtype or self.rt.dtype)
        if out is None:
            out = b.reg(self.out_features, dt)
        b.op(OP_LINEAR, in0=x, out0=out, w=b.ptr(self.weight), bias=b.ptr(self.bias), w_dtype=_dt(self.weight.dtype),
             ldw=self.weight.stride(0), n=self.out_features, k=self.in_features, out_dtype=dt)
        return out


class JoinedLinear(Part):
    """Several matrices with the same output applied to inputs laid side by side: y = [x1 | x2 | ...]
    [W1 | W2 | ...]^T (+ b1 + b2 ...).  The sum of the products x_i W_i^T is then taken inside one
    product's 32-bit accumulators and rounded once: how a block whose sublayers run side by side adds
    its mixer's and its feed-forward's outputs.  `pieces`: (weight tensor name, in features, bias
    tensor name or None); `offsets[i]` is where piece i's inputs start in a row of x.  `bias_scales`: what each piece's
    bias is multiplied by, in 32-bit (a block that scales its sublayers scales their inputs here and their biases so)."""

    def __init__(self, out_features: int, pieces, bias_scales=None):
        self.out_features = int(out_features)
        self.bias_scales = [1.0] * len(pieces) if bias_scales is None else [float(s) for s in bias_scales]
        self.pieces = [(w, int(k), b) for w, k, b in pieces]
        self.offsets, at = [], 0
        for _, k, _ in self.pieces:
            self.offsets.append(at)
            at += k
        self.in_features = at
        self.weight = None
        self.bias = None

    def own_weight_specs(self):
        specs = [WeightSpec(w, (self.out_features, k), "matrix") for w, k, _ in self.pieces]
        specs += [WeightSpec(b, (self.out_features,), "bias") for _, _, b in self.pieces if b is not None]
        return specs

    def bind_own(self, tensors, rt: Runtime):
        ws = [to_compute(tensors[w], rt) for w, _, _ in self.pieces]
        if len({w.dtype for w in ws}) > 1:
            ws = [w.float() for w in ws]
        self.weight = ws[0].contiguous() if len(ws) == 1 else torch.cat(ws, dim=1).contiguous()
        bs = [to_f32_vector(tensors[b], rt) * s if s != 1.0 else to_f32_vector(tensors[b], rt)
              for (_, _, b), s in zip(self.pieces, self.bias_scales) if b is not None]
        self.bias = None
        if bs:
            total = bs[0]
            for b in bs[1:]:
                total = total + b
            self.bias = total.contiguous()

    def weight_bytes(self):
        return self.weight.numel() * self.weight.element_size()

    def forward(self, x, out_dtype=None, skip: int = 0):
        """`skip`: x holds no inputs for the first that many columns, which the product leaves out."""
        w = self.weight[:, skip:] if skip else self.weight
        return self.rt.k.linear(x, w, self.bias, out_dtype or self.rt.dtype)


class BlockDiagonalLinear(Part):
    """Several matrices applied side by side, each to its own run of inputs: y = [W1 x1 | W2 x2 | ...] for x = [x1 | x2 |
    ...], as one product with the matrices on the diagonal of a larger one (zeros elsewhere).  For the second halves
    of low-rank projections, whose inputs are so narrow that one launch is worth more than the zeros cost.  `pieces`:
    (weight tensor name, out features, in features); the in features may be `FreeDim`s.  `in_features` and
    `out_features` are those of the whole once it is bound."""

    def __init__(self, pieces):
        self.pieces = list(pieces)
        self.in_features = sum(k for _, _, k in self.pieces)
        self.out_features = sum(o for _, o, _ in self.pieces)
        self.weight = None

    def own_weight_specs(self):
        return [WeightSpec(n, (o, k), "matrix") for n, o, k in self.pieces]

    def bind_own(self, tensors, rt: Runtime):
        ws = [to_compute(tensors[n], rt) for n, _, _ in self.pieces]
        if len({w.dtype for w in ws}) > 1:
            ws = [w.float() for w in ws]
        self.weight = ws[0].contiguous() if len(ws) == 1 else torch.block_diag(*ws).contiguous()
        self.out_features, self.in_features = self.weight.shape

    def weight_bytes(self):
        return self.weight.numel() * self.weight.element_size()

    def forward(self, x, out_dtype=None):
        return self.rt.k.linear(x, self.weight, None, out_dtype or self.rt.dtype)
