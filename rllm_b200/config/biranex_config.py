"""Typed configuration of the Biranex decoder, read from ``config.json``.

A Biranex model is a list of layers whose sublayers read the stream itself and
are normalised on their way back into it.  Each layer has a mixer of one of two
kinds and a dense feed-forward or none.  Keys:

    architecture: "Biranex"      vocab, width, residual_mult        norm: {eps}
    layers: [{type, mixer: {...}, mlp: {kind: "dense", ff} | null}, ...]
      type "channel_delta": mixer {heads, kv_heads, dim, vdim, conv}
      type "parallel":      mixer {left:  {heads, kv_heads, dim, vdim, scale, mask: {size},
                                           rot: {base, dims, scaling: {factor} | absent}},
                                   left_scale,
                                   right: {heads, vdim, state, groups, conv, norm_groups},
                                   right_scale}

Every size and constant is taken from these keys (the ranks of the low-rank
pairs of a channel_delta mixer are the tensors' own); optional
``max_positions`` (default 131,072) bounds a request's length for the engine,
which sizes its cache pools by it (the design itself has no bound).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .model_config import ConfigError

MIXER_KINDS = ("channel_delta", "parallel")
MLP_KINDS = ("dense",)


@dataclass(frozen=True)
class DeltaMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass(frozen=True)
class RotatedWindowAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int]             # None: no window
    rot_base: float
    rot_dims: int                     # 0: nothing rotates
    rot_factor: float


@dataclass(frozen=True)
class StateSpaceMixer:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int


@dataclass(frozen=True)
class ScaledParallel:
    left: RotatedWindowAttention
    left_scale: float
    right: StateSpaceMixer
    right_scale: float


@dataclass(frozen=True)
class BiranexLayer:
    kind: str
    mixer: object
    ff: Optional[int]                 # the dense feed-forward's inner size; None: no feed-forward


@dataclass(frozen=True)
class BiranexConfig:
    vocab: int
    width: int
    eps: float
    residual_mult: float
    layers: Tuple[BiranexLayer, ...]
    max_positions: int = 1 << 17
    torch_dtype: str = "bfloat16"

    @staticmethod
    def from_json(raw: Mapping[str, Any]) -> "BiranexConfig":
        def need(d: Mapping[str, Any], key: str, where: str):
            if not isinstance(d, Mapping) or key not in d:
                raise ConfigError(f"config.json: {where} lacks {key!r}")
            return d[key]

        def positive(d, key, where) -> int:
            v = int(need(d, key, where))
            if v < 1:
                raise ConfigError(f"config.json: {where}.{key} must be positive")
            return v

        def whole_groups(where, what, total, per, parts):
            if total % parts:
                raise ConfigError(f"config.json: {where}: {what} {total} is no multiple of {per} {parts}")

        raw_layers = need(raw, "layers", "the configuration")
        if not isinstance(raw_layers, (list, tuple)) or not raw_layers:
            raise ConfigError("config.json: layers must be a non-empty list")
        layers = []
        for i, L in enumerate(raw_layers):
            where = f"layers[{i}]"
            kind = str(need(L, "type", where))
            if kind not in MIXER_KINDS:
                raise ConfigError(f"config.json: {where} has mixer type {kind!r}; known: {list(MIXER_KINDS)}")
            m, mw = need(L, "mixer", where), where + ".mixer"
            if kind == "channel_delta":
                mixer = DeltaMixer(*(positive(m, k, mw) for k in ("heads", "kv_heads", "dim", "vdim", "conv")))
                whole_groups(mw, "heads", mixer.heads, "kv_heads", mixer.kv_heads)
            else:
                a, aw = need(m, "left", mw), mw + ".left"
                rot, mask = a.get("rot"), a.get("mask")
                base, dims, factor = 1.0, 0, 1.0
                if rot is not None:
                    base, dims = float(need(rot, "base", aw + ".rot")), int(need(rot, "dims", aw + ".rot"))
                    scaling = rot.get("scaling")
                    if scaling is not None:
                        factor = float(need(scaling, "factor", aw + ".rot.scaling"))
                    if factor <= 0 or base <= 0:
                        raise ConfigError(f"config.json: {aw}.rot: base and scaling.factor must be positive")
                left = RotatedWindowAttention(
                    positive(a, "heads", aw), positive(a, "kv_heads", aw), positive(a, "dim", aw),
                    positive(a, "vdim", aw), float(need(a, "scale", aw)),
                    positive(mask, "size", aw + ".mask") if mask is not None else None, base, dims, factor)
                whole_groups(aw, "heads", left.heads, "kv_heads", left.kv_heads)
                if dims % 2 or not 0 <= dims <= left.dim:
                    raise ConfigError(f"config.json: {aw}.rot.dims {dims} must be even and within dim {left.dim}")
                b, bw = need(m, "right", mw), mw + ".right"
                right = StateSpaceMixer(*(positive(b, k, bw) for k in ("heads", "vdim", "state", "groups", "conv",
                                                                       "norm_groups")))
                whole_groups(bw, "heads", right.heads, "groups", right.groups)
                whole_groups(bw, "heads * vdim", right.heads * right.vdim, "norm_groups", right.norm_groups)
                mixer = ScaledParallel(left, float(need(m, "left_scale", mw)), right,
                                       float(need(m, "right_scale", mw)))
            mlp, ff = L.get("mlp"), None
            if mlp is not None:
                fw = where + ".mlp"
                if str(need(mlp, "kind", fw)) not in MLP_KINDS:
                    raise ConfigError(f"config.json: {fw}.kind {mlp['kind']!r}; known: {list(MLP_KINDS)}")
                ff = positive(mlp, "ff", fw)
            layers.append(BiranexLayer(kind, mixer, ff))
        return BiranexConfig(vocab=positive(raw, "vocab", "the configuration"),
                             width=positive(raw, "width", "the configuration"),
                             eps=float(need(need(raw, "norm", "the configuration"), "eps", "norm")),
                             residual_mult=float(need(raw, "residual_mult", "the configuration")),
                             layers=tuple(layers), max_positions=int(raw.get("max_positions", 1 << 17)),
                             torch_dtype=str(raw.get("torch_dtype", "bfloat16")))
