"""Bikovik as a ``ModelSpec``: a decoder of ``pre_norm`` layers with dynamic-tanh norms whose mixers are of three
kinds:

``attention``  windowed grouped-query attention with kept first tokens, biases on queries, keys and values,
               talking heads (every head's scores are a learned mixture of all heads' scores) and, in some layers,
               values mixed with those of the first such layer.
``hgrn2``      linear attention with a decay per key channel, one minus which is the key.
``retention``  linear attention with a fixed decay per head, rotated queries and keys and a SiLU gate.

The feed-forward is dense and gated, with both factors clamped, or absent.  The embedding is multiplied by a
constant; the logits are the head's, capped by a tanh.

Tensor names: ``embed``, ``head``, ``final.norm``, and per layer ``l<i>.`` + ``norm1|norm2`` (every norm with
``.alpha`` and ``.b`` beside its weight), ``mix.*`` (attention: q, k, v with ``.b``, vmix, talk, o; hgrn2: q, f, f.b,
lower, v, norm, o; retention: q, k, v, g, o) and ``mlp.*`` (gate, up, down).
"""
from __future__ import annotations

from ..config.bikovik_config import BikovikConfig
from ..config.registry import register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, Run

GATE_SLOPE, UP_SHIFT = 1.702, 1.0   # of the feed-forward's gate: g sigmoid(slope g) (u + shift)


def _norm(size: int, name: str) -> PartSpec:
    return PartSpec.of("dynamic_tanh", size=size, name=name, alpha_name=name + ".alpha", shift_name=name + ".b")


def _rotary(rot, dim: int):
    return None if rot is None else PartSpec.of("rotary", head_dim=dim, rotary_dim=rot.dims, theta=rot.base)


def bikovik_spec(cfg: BikovikConfig) -> ModelSpec:
    H = cfg.width
    layers, values_seen = [], False
    for i, L in enumerate(cfg.layers):
        m = L.mixer
        if L.kind == "attention":
            mix = None
            if m.v_mix:
                mix, values_seen = ("mixed" if values_seen else "source"), True
            names = {k: k for k in ("q", "k", "v", "o")}
            names.update(q_bias="q.b", k_bias="k.b", v_bias="v.b", talk="talk", value_mix="vmix")
            mixer = PartSpec.of("attention", hidden_size=H, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim,
                                v_dim=m.vdim, window=m.window, keep_first=m.keep_first if m.window else 0, scale=m.scale,
                                position=_rotary(m.rot, m.dim), bias="qkv", head_mix=True, value_mix=mix,
                                tensor_prefix="mix.", tensor_names=names)
        elif L.kind == "hgrn2":
            names = {k: k for k in ("q", "f", "v", "norm", "o", "lower")}
            mixer = PartSpec.of("hgrn2", hidden_size=H, num_heads=m.heads, head_dim=m.dim, v_dim=m.vdim, eps=cfg.eps,
                                tensor_prefix="mix.", tensor_names=dict(names, f_bias="f.b"))
        else:
            mixer = PartSpec.of("retention", hidden_size=H, num_heads=m.heads, head_dim=m.dim, v_dim=m.vdim,
                                decay=m.decay, position=_rotary(m.rot, m.dim), eps=cfg.eps, tensor_prefix="mix.",
                                tensor_names={k: k for k in ("q", "k", "v", "g", "o")})
        ffn = None
        if L.mlp is not None:
            ffn = PartSpec.of("gated_mlp", hidden_size=H, intermediate_size=L.mlp.ff, activation="silu",
                              limit=L.mlp.limit, slope=GATE_SLOPE, up_shift=UP_SHIFT, tensor_prefix="mlp.",
                              tensor_names={"gate": "gate", "up": "up", "down": "down"})
        layers.append(LayerSpec(block="pre_norm", mixer=mixer, ffn=ffn, norms=(_norm(H, "norm1"), _norm(H, "norm2")),
                                prefix=f"l{i}."))
    return ModelSpec(
        hidden_size=H, vocab_size=cfg.vocab,
        embedding=PartSpec.of("token_embedding", vocab_size=cfg.vocab, hidden_size=H, name="embed",
                              scale=cfg.embedding_scale),
        layers=tuple(layers), order=tuple(Run(layer=i, cache=i) for i in range(len(layers))),
        final_norm=_norm(H, "final.norm"),
        head=PartSpec.of("lm_head", vocab_size=cfg.vocab, hidden_size=H, name="head", softcap=cfg.logit_softcap),
        max_positions=cfg.max_positions)


register_architecture("Bikovik", BikovikConfig.from_json, bikovik_spec)
