"""Typed configuration of the Bikovik decoder, read from ``config.json``.

A Bikovik model is a list of pre-norm layers (dynamic-tanh norms), each with a
mixer of one of three kinds and a dense feed-forward or none.  Keys:

    architecture: "Bikovik"      vocab, width, logit_softcap | absent
    embedding: {scale}           norm: {eps}
    layers: [{type, mixer: {...}, mlp: {kind: "dense", ff, limit} | null}, ...]
      type "attention": mixer {heads, kv_heads, dim, vdim, scale, rot: {base, dims} | absent,
                               mask: {size, keep_first} | absent, v_mix}
      type "hgrn2":     mixer {heads, dim, vdim}
      type "retention": mixer {heads, dim, vdim, decay: [a number a head], rot: {base, dims} | absent}

Every size and constant is taken from these keys; optional ``max_positions``
(default 131,072) bounds a request's length for the engine, which sizes its
cache pools by it (the design itself has no bound).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .model_config import ConfigError

MIXER_KINDS = ("attention", "hgrn2", "retention")
MLP_KINDS = ("dense",)


@dataclass(frozen=True)
class Rotation:
    base: float
    dims: int


@dataclass(frozen=True)
class TalkingAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[Rotation]
    window: Optional[int]             # None: every earlier key is visible
    keep_first: int
    v_mix: bool


@dataclass(frozen=True)
class Hgrn2:
    heads: int
    dim: int
    vdim: int


@dataclass(frozen=True)
class Retention:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    rot: Optional[Rotation]


@dataclass(frozen=True)
class ClampedMlp:
    ff: int
    limit: float


@dataclass(frozen=True)
class BikovikLayer:
    kind: str
    mixer: object
    mlp: Optional[ClampedMlp]         # None: no feed-forward


@dataclass(frozen=True)
class BikovikConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    logit_softcap: Optional[float]
    layers: Tuple[BikovikLayer, ...]
    max_positions: int = 1 << 17
    torch_dtype: str = "bfloat16"

    @staticmethod
    def from_json(raw: Mapping[str, Any]) -> "BikovikConfig":
        def need(d: Mapping[str, Any], key: str, where: str):
            if not isinstance(d, Mapping) or key not in d:
                raise ConfigError(f"config.json: {where} lacks {key!r}")
            return d[key]

        def positive(d, key, where) -> int:
            v = int(need(d, key, where))
            if v < 1:
                raise ConfigError(f"config.json: {where}.{key} must be positive")
            return v

        def rotation(m, dim: int, where) -> Optional[Rotation]:
            rot = m.get("rot")
            if rot is None:
                return None
            base, dims = float(need(rot, "base", where + ".rot")), int(need(rot, "dims", where + ".rot"))
            if dims % 2 or not 0 <= dims <= dim:
                raise ConfigError(f"config.json: {where}.rot.dims {dims} must be even and within dim {dim}")
            if not base > 0:
                raise ConfigError(f"config.json: {where}.rot.base must be positive")
            return Rotation(base, dims) if dims else None

        raw_layers = need(raw, "layers", "the configuration")
        if not isinstance(raw_layers, (list, tuple)) or not raw_layers:
            raise ConfigError("config.json: layers must be a non-empty list")
        layers, first_values = [], None
        for i, L in enumerate(raw_layers):
            where = f"layers[{i}]"
            kind = str(need(L, "type", where))
            if kind not in MIXER_KINDS:
                raise ConfigError(f"config.json: {where} has mixer type {kind!r}; known: {list(MIXER_KINDS)}")
            m, mw = need(L, "mixer", where), where + ".mixer"
            heads, dim, vdim = (positive(m, k, mw) for k in ("heads", "dim", "vdim"))
            if kind == "attention":
                kv, mask = positive(m, "kv_heads", mw), m.get("mask")
                if heads % kv:
                    raise ConfigError(f"config.json: {mw}: heads {heads} is no multiple of kv_heads {kv}")
                keep = int(mask.get("keep_first") or 0) if mask is not None else 0
                if keep < 0:
                    raise ConfigError(f"config.json: {mw}.mask.keep_first must not be negative")
                mixer = TalkingAttention(heads, kv, dim, vdim, float(need(m, "scale", mw)), rotation(m, dim, mw),
                                         positive(mask, "size", mw + ".mask") if mask is not None else None, keep,
                                         bool(m.get("v_mix", False)))
                if mixer.v_mix:
                    first_values = first_values or (i, kv, vdim)
                    if (kv, vdim) != first_values[1:]:
                        raise ConfigError(f"config.json: {mw}.v_mix: kv_heads {kv} and vdim {vdim} differ from those of "
                                          f"layers[{first_values[0]}], whose values are mixed in")
            elif kind == "hgrn2":
                mixer = Hgrn2(heads, dim, vdim)
            else:
                decay = tuple(float(x) for x in need(m, "decay", mw))
                if len(decay) != heads:
                    raise ConfigError(f"config.json: {mw}.decay has {len(decay)} numbers for {heads} heads")
                if any(not 0.0 <= x <= 1.0 for x in decay):
                    raise ConfigError(f"config.json: {mw}.decay: numbers from 0 to 1")
                mixer = Retention(heads, dim, vdim, decay, rotation(m, dim, mw))
            mlp, ff = L.get("mlp"), None
            if mlp is not None:
                fw = where + ".mlp"
                if str(need(mlp, "kind", fw)) not in MLP_KINDS:
                    raise ConfigError(f"config.json: {fw}.kind {mlp['kind']!r}; known: {list(MLP_KINDS)}")
                ff = ClampedMlp(positive(mlp, "ff", fw), float(need(mlp, "limit", fw)))
                if not ff.limit > 0:
                    raise ConfigError(f"config.json: {fw}.limit must be positive")
            layers.append(BikovikLayer(kind, mixer, ff))
        cap = raw.get("logit_softcap")
        if cap is not None and not float(cap) > 0:
            raise ConfigError("config.json: logit_softcap must be positive")
        return BikovikConfig(vocab=positive(raw, "vocab", "the configuration"),
                             width=positive(raw, "width", "the configuration"),
                             eps=float(need(need(raw, "norm", "the configuration"), "eps", "norm")),
                             embedding_scale=float(need(need(raw, "embedding", "the configuration"), "scale", "embedding")),
                             logit_softcap=None if cap is None else float(cap), layers=tuple(layers),
                             max_positions=int(raw.get("max_positions", 1 << 17)),
                             torch_dtype=str(raw.get("torch_dtype", "bfloat16")))
