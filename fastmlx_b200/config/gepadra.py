"""Typed configuration of the Gepadra design, read from config.json.

A Gepadra model is a list of parallel layers with two norms (weights stored around zero): x <- x + (mixer(N1(x)) + ff(N2(x))).
The mixer is one of

* `attention`: grouped-query softmax attention with biases, half-split rotary positions on the heads' first dimensions, a
  sliding window beside which a request's first tokens stay visible, a learned term per head in the softmax's denominator,
  and (`v_mix`) values mixed with those of the first layer that mixes;
* `mlstm`: a matrix memory with exponential input and forget gates (capped), a normaliser and a running maximum.

The feed-forward is dense and gated (clamped), a mixture of experts without a gate whose inputs are weighed by sigmoid
scores (with an optional shared expert behind a sigmoid gate), or absent.  The output head is the embedding table.  Every size
and constant stands in config.json; what it does not name does not exist (no rot: nothing is rotated; no mask: every earlier
key is seen; no shared: no shared expert).
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any, Mapping

from .base import ConfigError, ModelConfig


def _int(d: Mapping, key: str, where: str, low: int = 1) -> int:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, (int, float)) or int(v) != v or int(v) < low:
        raise ConfigError(f"gepadra: {where}.{key} must be an integer >= {low}, got {v!r}")
    return int(v)


def _float(d: Mapping, key: str, where: str, positive: bool = False) -> float:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, (int, float)) or not math.isfinite(float(v)) or (positive and not v > 0):
        raise ConfigError(f"gepadra: {where}.{key} must be a finite{' positive' if positive else ''} number, got {v!r}")
    return float(v)


def _block(d: Mapping, key: str, where: str) -> Mapping:
    """An optional sub-object; absent or null is empty."""
    v = d.get(key)
    if v is None:
        return {}
    if not isinstance(v, Mapping):
        raise ConfigError(f"gepadra: {where}.{key} must be an object")
    return v


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int                   # 0: every earlier token is seen
    keep_first: int               # beside a window: the first tokens that stay visible
    rot_dims: int                 # 0: no rotation
    rot_base: float
    v_mix: bool

    @staticmethod
    def from_dict(d: Mapping[str, Any], where: str) -> "AttentionConfig":
        mask, rot = _block(d, "mask", where), _block(d, "rot", where)
        dim = _int(d, "dim", where)
        dims = _int(rot, "dims", where + ".rot", 0) if rot else 0
        if dims % 2 or dims > dim:
            raise ConfigError(f"gepadra: {where}.rot.dims must be even and at most {dim}, got {dims}")
        v_mix = d.get("v_mix", False)
        if not isinstance(v_mix, bool):
            raise ConfigError(f"gepadra: {where}.v_mix must be true or false, got {v_mix!r}")
        c = AttentionConfig(
            _int(d, "heads", where), _int(d, "kv_heads", where), dim, _int(d, "vdim", where), _float(d, "scale", where),
            _int(mask, "size", where + ".mask") if mask else 0,
            _int(mask, "keep_first", where + ".mask", 0) if mask.get("keep_first") is not None else 0,
            dims, _float(rot, "base", where + ".rot", True) if dims else 1.0, v_mix)
        if c.heads % c.kv_heads:
            raise ConfigError(f"gepadra: {where}: {c.heads} heads are no multiple of {c.kv_heads} kv_heads")
        if c.dim > 256:
            raise ConfigError(f"gepadra: {where}: a head size up to 256, got {c.dim}")
        return c


@dataclass(frozen=True)
class MatrixMemoryConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @staticmethod
    def from_dict(d: Mapping[str, Any], where: str) -> "MatrixMemoryConfig":
        c = MatrixMemoryConfig(_int(d, "heads", where), _int(d, "dim", where), _int(d, "vdim", where),
                               _float(d, "gate_cap", where, True))
        if c.dim > 512:
            raise ConfigError(f"gepadra: {where}: a key size up to 512, got {c.dim}")
        return c


@dataclass(frozen=True)
class DenseMlpConfig:
    ff: int
    limit: float
    kind: str = "dense"


@dataclass(frozen=True)
class ExpertsMlpConfig:
    experts: int
    top: int
    ff: int
    shared_ff: int                # 0: no shared expert
    kind: str = "moe"


def _mlp(m, where: str) -> DenseMlpConfig | ExpertsMlpConfig | None:
    if m is None:
        return None
    if not isinstance(m, Mapping) or m.get("kind") not in ("dense", "moe"):
        raise ConfigError(f"gepadra: {where} must be null or an object of kind 'dense' or 'moe', got {m!r}")
    if m["kind"] == "dense":
        c = DenseMlpConfig(_int(m, "ff", where), _float(m, "limit", where))
        if c.limit < 0:
            raise ConfigError(f"gepadra: {where}.limit must not be negative, got {c.limit}")
        return c
    router, expert, shared = (_block(m, k, where) for k in ("router", "expert", "shared"))
    c = ExpertsMlpConfig(_int(router, "experts", where + ".router"), _int(router, "top", where + ".router"),
                         _int(expert, "ff", where + ".expert"), _int(shared, "ff", where + ".shared") if shared else 0)
    if c.top > c.experts:
        raise ConfigError(f"gepadra: {where}.router: top={c.top} of {c.experts} experts")
    return c


@dataclass(frozen=True)
class LayerConfig:
    type: str                     # "attention" | "mlstm"
    mixer: AttentionConfig | MatrixMemoryConfig
    mlp: DenseMlpConfig | ExpertsMlpConfig | None


_MIXERS = {"attention": AttentionConfig, "mlstm": MatrixMemoryConfig}


@dataclass(frozen=True)
class GepadraConfig(ModelConfig):
    vocab: int = 0
    width: int = 0
    layers: tuple[LayerConfig, ...] = ()
    norm_eps: float = 0.0
    raw: tuple = ()               # the config.json items as read, for to_dict

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def eos_token_id(self) -> int:
        return -1

    @property
    def first_v_mix(self) -> int | None:
        """The layer whose values the later mixing layers mix in."""
        return next((i for i, s in enumerate(self.layers) if s.type == "attention" and s.mixer.v_mix), None)

    @staticmethod
    def from_dict(c: Mapping[str, Any]) -> "GepadraConfig":
        layers = c.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("gepadra: `layers` must be a list with at least one layer")
        out = []
        for i, spec in enumerate(layers):
            where = f"layers[{i}]"
            if not isinstance(spec, Mapping) or not isinstance(spec.get("mixer"), Mapping):
                raise ConfigError(f"gepadra: {where} must be an object with a `mixer`")
            kind = spec.get("type")
            if kind not in _MIXERS:
                raise ConfigError(f"gepadra: {where}.type must be one of {sorted(_MIXERS)}, got {kind!r}")
            out.append(LayerConfig(kind, _MIXERS[kind].from_dict(spec["mixer"], where + ".mixer"), _mlp(spec.get("mlp"), where + ".mlp")))
        norm = c.get("norm")
        if not isinstance(norm, Mapping):
            raise ConfigError("gepadra: `norm` must be an object with `eps`")
        eps = _float(norm, "eps", "norm")
        if eps < 0:
            raise ConfigError(f"gepadra: norm.eps must not be negative, got {eps}")
        cfg = GepadraConfig(vocab=_int(c, "vocab", "config"), width=_int(c, "width", "config"), layers=tuple(out), norm_eps=eps,
                            raw=tuple(sorted(c.items(), key=lambda kv: kv[0])))
        mixing = [(i, s.mixer.kv_heads * s.mixer.vdim) for i, s in enumerate(out) if s.type == "attention" and s.mixer.v_mix]
        if len({n for _, n in mixing}) > 1:
            raise ConfigError(f"gepadra: layers that mix their values need equally many per token, got {mixing}")
        return cfg

    def to_dict(self) -> dict:
        return dict(self.raw)
