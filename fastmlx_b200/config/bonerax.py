"""Typed configuration of the Bonerax design, read from config.json.

A Bonerax model is a list of layers whose sublayers read the stream itself and are normed on their way out: x <- x +
L1(mixer(x)), then x <- x + L2(ff(x)), every L a layer norm with a weight and no bias.  The mixer is one of

* `gla`: gated linear attention, a matrix of 32-bit state per head whose rows decay by sigmoid(.)^(1/tau) per channel;
* `channel_delta`: the delta rule with a decay per head and key channel, behind short causal convolutions;
* `parallel`: left_scale * left + right_scale * right on the same input, left a sliding-window softmax attention (q and k
  RMS-normed per head, interleaved rotary positions optionally with YaRN's rescaled frequencies, biases), right a
  `channel_delta`.

The feed-forward is dense and gated (SiLU), a mixture of such experts (the largest biased logits choose, the softmax
over the chosen logits weighs), or absent.  A layer with `weights_of` uses another layer's tensors with a cache and a
state of its own.  The logits are multiplied by `logit_scale` and capped by `logit_softcap`.  Every size and constant
stands in config.json but the ranks of the low-rank projections, which the tensors give; what it does not name does not
exist (no rot: nothing is rotated; no scaling: frequencies as they stand; no mask: every earlier key is seen; no
logit_softcap: logits are not capped).
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any, Mapping

from .base import ConfigError, ModelConfig
from .llama import YarnScaling


def _int(d: Mapping, key: str, where: str, low: int = 1) -> int:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, (int, float)) or int(v) != v or int(v) < low:
        raise ConfigError(f"bonerax: {where}.{key} must be an integer >= {low}, got {v!r}")
    return int(v)


def _float(d: Mapping, key: str, where: str) -> float:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, (int, float)) or not math.isfinite(float(v)):
        raise ConfigError(f"bonerax: {where}.{key} must be a finite number, got {v!r}")
    return float(v)


def _object(d: Mapping, key: str, where: str) -> Mapping:
    v = d.get(key)
    if not isinstance(v, Mapping):
        raise ConfigError(f"bonerax: {where}.{key} must be an object, got {v!r}")
    return v


@dataclass(frozen=True)
class WindowedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int                   # 0: every earlier key is seen
    rot_dims: int                 # 0: no rotation
    rot_base: float
    scaling: YarnScaling | None

    @staticmethod
    def from_dict(d: Mapping[str, Any], where: str) -> "WindowedAttentionConfig":
        dim = _int(d, "dim", where)
        dims, base, scaling = 0, 1.0, None
        if d.get("rot") is not None:
            rot = _object(d, "rot", where)
            w = where + ".rot"
            dims = _int(rot, "dims", w, 0)
            if dims % 2 or dims > dim:
                raise ConfigError(f"bonerax: {w}.dims must be even and at most {dim}, got {dims}")
            if dims:
                base = _float(rot, "base", w)
                if base <= 0:
                    raise ConfigError(f"bonerax: {w}.base must be positive, got {base}")
            if dims and rot.get("scaling") is not None:
                sc = _object(rot, "scaling", w)
                w += ".scaling"
                scaling = YarnScaling(*(_float(sc, key, w) for key in ("factor", "original", "fast", "slow")))
                if min(scaling.factor, scaling.original, scaling.fast, scaling.slow) <= 0 or base == 1.0:
                    raise ConfigError(f"bonerax: {w}: factor, original, fast and slow must be positive, and rot.base not 1")
        window = _int(_object(d, "mask", where), "size", where + ".mask") if d.get("mask") is not None else 0
        c = WindowedAttentionConfig(_int(d, "heads", where), _int(d, "kv_heads", where), dim, _int(d, "vdim", where),
                                    _float(d, "scale", where), window, dims, base, scaling)
        if c.heads % c.kv_heads:
            raise ConfigError(f"bonerax: {where}: {c.heads} heads are no multiple of {c.kv_heads} kv_heads")
        if c.dim > 256 or c.vdim > 512:
            raise ConfigError(f"bonerax: {where}: keys up to 256 and values up to 512 wide, got {c.dim} and {c.vdim}")
        return c


@dataclass(frozen=True)
class ChannelDeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int                     # taps of the short convolutions

    @staticmethod
    def from_dict(d: Mapping[str, Any], where: str) -> "ChannelDeltaConfig":
        c = ChannelDeltaConfig(*(_int(d, key, where) for key in ("heads", "kv_heads", "dim", "vdim", "conv")))
        if c.heads % c.kv_heads:
            raise ConfigError(f"bonerax: {where}: {c.heads} heads are no multiple of {c.kv_heads} kv_heads")
        if c.dim > 512 or c.conv > 16:
            raise ConfigError(f"bonerax: {where}: up to 512 rows of state per column and 16 taps, got {c.dim} and {c.conv}")
        return c


@dataclass(frozen=True)
class GatedLinearConfig:
    heads: int
    dim: int
    vdim: int
    tau: float

    @staticmethod
    def from_dict(d: Mapping[str, Any], where: str) -> "GatedLinearConfig":
        c = GatedLinearConfig(*(_int(d, key, where) for key in ("heads", "dim", "vdim")), _float(d, "tau", where))
        if c.dim > 512 or c.tau <= 0:
            raise ConfigError(f"bonerax: {where}: up to 512 rows of state per column and a positive tau, got {c.dim} and {c.tau}")
        return c


@dataclass(frozen=True)
class ParallelConfig:
    left: WindowedAttentionConfig
    right: ChannelDeltaConfig
    left_scale: float
    right_scale: float

    @staticmethod
    def from_dict(d: Mapping[str, Any], where: str) -> "ParallelConfig":
        return ParallelConfig(WindowedAttentionConfig.from_dict(_object(d, "left", where), where + ".left"),
                              ChannelDeltaConfig.from_dict(_object(d, "right", where), where + ".right"),
                              _float(d, "left_scale", where), _float(d, "right_scale", where))


@dataclass(frozen=True)
class DenseMlpConfig:
    ff: int


@dataclass(frozen=True)
class ExpertsMlpConfig:
    experts: int
    top: int
    ff: int


@dataclass(frozen=True)
class LayerConfig:
    type: str
    mixer: ParallelConfig | ChannelDeltaConfig | GatedLinearConfig
    mlp: DenseMlpConfig | ExpertsMlpConfig | None
    weights_of: int               # the layer whose tensors this one uses (its own number where it has its own)


_MIXERS = {"parallel": ParallelConfig, "channel_delta": ChannelDeltaConfig, "gla": GatedLinearConfig}


def _mlp(d: Mapping, where: str) -> DenseMlpConfig | ExpertsMlpConfig | None:
    if d.get("mlp") is None:
        return None
    mlp, where = _object(d, "mlp", where), where + ".mlp"
    if mlp.get("kind") == "dense":
        return DenseMlpConfig(_int(mlp, "ff", where))
    if mlp.get("kind") != "moe":
        raise ConfigError(f"bonerax: {where}.kind must be 'dense' or 'moe', got {mlp.get('kind')!r}")
    router = _object(mlp, "router", where)
    c = ExpertsMlpConfig(_int(router, "experts", where + ".router"), _int(router, "top", where + ".router"),
                         _int(_object(mlp, "expert", where), "ff", where + ".expert"))
    if c.top > c.experts:
        raise ConfigError(f"bonerax: {where}: top={c.top} of {c.experts} experts")
    return c


@dataclass(frozen=True)
class BoneraxConfig(ModelConfig):
    vocab: int = 0
    width: int = 0
    layers: tuple[LayerConfig, ...] = ()
    norm_eps: float = 0.0
    logit_scale: float = 1.0
    logit_softcap: float = 0.0    # 0: logits are not capped
    raw: tuple = ()               # the config.json items as read, for to_dict

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def eos_token_id(self) -> int:
        return -1

    @staticmethod
    def from_dict(c: Mapping[str, Any]) -> "BoneraxConfig":
        layers = c.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("bonerax: `layers` must be a list with at least one layer")
        out = []
        for i, spec in enumerate(layers):
            where = f"layers[{i}]"
            if not isinstance(spec, Mapping):
                raise ConfigError(f"bonerax: {where} must be an object")
            kind = spec.get("type")
            if kind not in _MIXERS:
                raise ConfigError(f"bonerax: {where}.type must be one of {sorted(_MIXERS)}, got {kind!r}")
            own = i if spec.get("weights_of") is None else _int(spec, "weights_of", where, 0)
            if own >= len(layers):
                raise ConfigError(f"bonerax: {where}.weights_of names layer {own} of {len(layers)}")
            out.append(LayerConfig(kind, _MIXERS[kind].from_dict(_object(spec, "mixer", where), where + ".mixer"), _mlp(spec, where), own))
        for i, layer in enumerate(out):               # a chain of names ends at a layer with tensors of its own
            own, steps = layer.weights_of, 0
            while out[own].weights_of != own and steps <= len(out):
                own, steps = out[own].weights_of, steps + 1
            source = out[own]
            if steps > len(out) or (source.type, source.mixer, source.mlp) != (layer.type, layer.mixer, layer.mlp):
                raise ConfigError(f"bonerax: layers[{i}].weights_of: layer {own} is not of the same kind and sizes")
            out[i] = LayerConfig(layer.type, layer.mixer, layer.mlp, own)
        eps = _float(_object(c, "norm", "config"), "eps", "norm")
        if eps < 0:
            raise ConfigError(f"bonerax: norm.eps must not be negative, got {eps}")
        cap = _float(c, "logit_softcap", "config") if c.get("logit_softcap") is not None else 0.0
        if cap < 0:
            raise ConfigError(f"bonerax: logit_softcap must not be negative, got {cap}")
        return BoneraxConfig(vocab=_int(c, "vocab", "config"), width=_int(c, "width", "config"), layers=tuple(out), norm_eps=eps,
                             logit_scale=_float(c, "logit_scale", "config") if c.get("logit_scale") is not None else 1.0,
                             logit_softcap=cap, raw=tuple(sorted(c.items(), key=lambda kv: kv[0])))

    def to_dict(self) -> dict:
        return dict(self.raw)
