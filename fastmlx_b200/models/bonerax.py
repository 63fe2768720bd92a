"""Bonerax, assembled from parts.

Every layer is a `PostNormBlock` (layer norms behind the sublayers, which read the stream itself) around a mixer and a
feed-forward, or the mixer alone.  The mixers: `GatedLinearAttention`; `ChannelDeltaMixer`; or a `PairMixer` that adds a
scaled `GQAAttention` on its route with 32-bit scores (q and k normed per head in front of an interleaved rotation with
YaRN's frequencies, biases, a sliding window) and a scaled `ChannelDeltaMixer`.  The feed-forward is a `SwiGLU` or a
`RoutedExperts` (SiLU experts, biased logits, weights over the chosen logits alone).  A layer with `weights_of` is a second
entry of the schedule for the same layer, with a cache and a state slot of its own.  Tensor names: `embed`,
`l<i>.norm1|norm2`, `l<i>.mix.<name>` (biases `<name>.b`, convolution taps `<name>.conv`; of a pair
`l<i>.mix.left.<name>` and `l<i>.mix.right.<name>`), `l<i>.mlp.gate|up|down` or `l<i>.mlp.router|router.b|e<j>.gate|up|down`,
`final.norm`, `head`; matrices are stored [out, in] under their bare names.
"""
from __future__ import annotations

from .. import registry
from ..config.bonerax import BoneraxConfig, DenseMlpConfig
from ..parts import (ChannelDeltaMixer, Embedding, GatedLinearAttention, GQAAttention, LayerNorm, LMHead, Model, NoPositionEncoding,
                     PairMixer, PostNormBlock, RotaryEmbedding, RoutedExperts, Run, SwiGLU)


def _channel_delta(m, width, eps, name, output):
    return ChannelDeltaMixer(width, m.heads, m.kv_heads, m.dim, m.vdim, m.conv, eps, name, output=output, weight_suffix="")


def _mixer(spec, width, eps, name):
    m = spec.mixer
    if spec.type == "gla":
        return GatedLinearAttention(width, m.heads, m.dim, m.vdim, m.tau, eps, name, weight_suffix="")
    if spec.type == "channel_delta":
        return _channel_delta(m, width, eps, name, True)
    a = m.left
    pos = RotaryEmbedding(a.dim, a.rot_base, scaling=a.scaling, traditional=True, rotary_dim=a.rot_dims) if a.rot_dims \
        else NoPositionEncoding()
    left = GQAAttention(width, a.heads, a.kv_heads, a.dim, pos, f"{name}.left", bias=True, late_bias=True, scale=a.scale,
                        window=a.window, proj_names=("q", "k", "v", "o"), v_head_dim=a.vdim, qk_norm_eps=eps,
                        qk_norm_weights=("q.norm", "k.norm"), qk_norm_first=True, output=False, weight_suffix="", bias_suffix=".b")
    return PairMixer(width, left, _channel_delta(m.right, width, eps, f"{name}.right", False), eps, name,
                     scales=(m.left_scale, m.right_scale))


def build_bonerax(cfg: BoneraxConfig) -> Model:
    d, eps = cfg.width, cfg.norm_eps
    embed = Embedding(cfg.vocab, d, "embed", suffix="")
    layers, place, drop = [], {}, []
    for i, spec in enumerate(cfg.layers):
        if spec.weights_of != i:
            continue
        p = f"l{i}"
        ffn = norm2 = None
        if spec.mlp is None:
            drop.append(f"{p}.norm2")                 # a layer without a feed-forward uses no second norm
        else:
            norm2 = LayerNorm(d, eps, f"{p}.norm2", suffix="")
            if isinstance(spec.mlp, DenseMlpConfig):
                ffn = SwiGLU(d, spec.mlp.ff, f"{p}.mlp", proj_names=("gate", "up", "down"), weight_suffix="")
            else:
                ffn = RoutedExperts(d, spec.mlp.experts, spec.mlp.top, spec.mlp.ff, 0.0, f"{p}.mlp", activation="silu",
                                    router_bias="router.b", weights="chosen")
        place[i] = len(layers)
        layers.append(PostNormBlock(_mixer(spec, d, eps, f"{p}.mix"), ffn, LayerNorm(d, eps, f"{p}.norm1", suffix=""), norm2))
    schedule = [Run(place[spec.weights_of]) for spec in cfg.layers]
    head = LMHead(cfg.vocab, d, "head", suffix="", scale=cfg.logit_scale, softcap=cfg.logit_softcap)
    return Model(embed, layers, LayerNorm(d, eps, "final.norm", suffix=""), head, schedule=schedule, vocab_size=cfg.vocab, drop=drop)


registry.register(["bonerax", "Bonerax"], BoneraxConfig.from_dict, build_bonerax, replace=True)
