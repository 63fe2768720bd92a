"""Gepadra, assembled from parts.

Every layer is a `ParallelBlock` with two norms (RMS norms whose weights are stored around zero, both of the same stream, in
one kernel) around a `GQAAttention` on its route with 32-bit scores (biases, partial rotary positions in the half-split
pairing, a window beside which the first tokens stay visible, a learned term per head in the denominator, values mixed with
those of the first mixing layer) or a `MatrixMemoryMixer`, and a `SwiGLU` with clamps, a `PlainRoutedExperts` (gelu experts
weighed on their inputs by sigmoid scores, a shared expert behind a gate) or no feed-forward.  Mixer and feed-forward hand on
their inner features, and one joined product takes both to the stream.  The head is tied to the embedding.  Tensor names:
`embed`, `l<i>.norm1|norm2`, `l<i>.mix.q|k|v|o` (biases `.b`), `l<i>.mix.sink|vmix`, `l<i>.mix.g|norm|i|f`,
`l<i>.mlp.gate|up|down` or `l<i>.mlp.router|e<j>.up|e<j>.down|shared.up|shared.down|shared.sg`, `final.norm`; matrices are
stored [out, in] under their bare names.
"""
from __future__ import annotations

from .. import registry
from ..config.gepadra import GepadraConfig
from ..parts import (Embedding, GQAAttention, LMHead, MatrixMemoryMixer, Model, NoPositionEncoding, ParallelBlock,
                     PlainRoutedExperts, RMSNorm, RotaryEmbedding, SwiGLU)


def build_gepadra(cfg: GepadraConfig) -> Model:
    d, eps = cfg.width, cfg.norm_eps
    embed = Embedding(cfg.vocab, d, "embed", suffix="")

    def norm(name):
        return RMSNorm(d, eps, name, offset=1.0, suffix="")

    layers, drop = [], []
    for i, spec in enumerate(cfg.layers):
        p, m = f"l{i}", spec.mixer
        if spec.type == "attention":
            pos = RotaryEmbedding(m.dim, m.rot_base, rotary_dim=m.rot_dims) if m.rot_dims else NoPositionEncoding()
            mix = None if not m.v_mix else "first" if i == cfg.first_v_mix else "later"
            mixer = GQAAttention(d, m.heads, m.kv_heads, m.dim, pos, f"{p}.mix", bias=True, scale=m.scale, window=m.window,
                                 keep_first=m.keep_first, proj_names=("q", "k", "v", "o"), v_head_dim=m.vdim, sink="sink",
                                 value_mix=mix, value_mix_name="vmix", output=False, out_bias=False, weight_suffix="",
                                 bias_suffix=".b")
            if mix is None:
                drop.append(f"{p}.mix.vmix")          # a layer that mixes nothing uses no share
        else:
            mixer = MatrixMemoryMixer(d, m.heads, m.dim, m.vdim, m.gate_cap, eps, f"{p}.mix", output=False, weight_suffix="")
        ffn = None
        if spec.mlp is None:
            drop.append(f"{p}.norm2")                 # a layer without a feed-forward uses no second norm
        elif spec.mlp.kind == "dense":
            ffn = SwiGLU(d, spec.mlp.ff, f"{p}.mlp", proj_names=("gate", "up", "down"), activation="clamped",
                         limit=spec.mlp.limit, output=False, weight_suffix="")
        else:
            e = spec.mlp
            ffn = PlainRoutedExperts(d, e.experts, e.top, e.ff, f"{p}.mlp", shared_ff=e.shared_ff, activation="gelu", correction=None,
                                     scores="sigmoid", weigh="input", output=False)
        layers.append(ParallelBlock(mixer, ffn, norm(f"{p}.norm1"), d, norm2=norm(f"{p}.norm2") if ffn is not None else None))
    head = LMHead(cfg.vocab, d, None, tied=embed)
    return Model(embed, layers, norm("final.norm"), head, vocab_size=cfg.vocab, drop=drop)


registry.register(["gepadra", "Gepadra"], GepadraConfig.from_dict, build_gepadra, replace=True)
