"""Biranex as a ``ModelSpec``: a decoder of ``post_norm`` layers (a sublayer reads the stream itself; its
result is RMS-normalised, multiplied by a constant and added) whose mixers are of two kinds:

``channel_delta``  the gated delta rule with a decay per key channel, short convolutions on queries, keys
                   and values, per-head norm and a low-rank output gate.
``parallel``       windowed grouped-query attention (queries and keys normalised over the whole projection,
                   rotation of pairs 2i, 2i + 1 at a lowered frequency, a learned sink and a sigmoid gate per
                   head) beside a ``state_space`` recurrence (Mamba-2: a scalar decay per head and token);
                   the result is a weighted sum of the two with constant weights.

The feed-forward is dense and SiLU-gated, or absent.  The output is the model's norm and the embedding
table as the head.

Tensor names: ``embed``, ``final.norm``, and per layer ``l<i>.`` + ``norm1|norm2``, ``mix.*``
(channel_delta: q, k, v, q.conv, k.conv, v.conv, b, a1, a2, A_log, dt_bias, norm, g1, g2, o; parallel:
left.q|k|v|o|g|sink, left.q.norm, left.k.norm, right.in|conv|conv.b|dt_bias|A_log|D|norm|o) and ``mlp.*``
(gate, up, down).
"""
from __future__ import annotations

from ..config.biranex_config import BiranexConfig
from ..config.registry import register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, Run

UNIT_EPS = 1e-6                     # under the root that makes queries and keys unit vectors


def _norm(size: int, eps: float, name: str) -> PartSpec:
    return PartSpec.of("rmsnorm", size=size, eps=eps, name=name)


def biranex_spec(cfg: BiranexConfig) -> ModelSpec:
    H = cfg.width
    layers = []
    for i, L in enumerate(cfg.layers):
        m = L.mixer
        if L.kind == "channel_delta":
            names = {k: k for k in ("q", "k", "v", "b", "a1", "a2", "dt_bias", "norm", "g1", "g2", "o")}
            names.update(q_conv="q.conv", k_conv="k.conv", v_conv="v.conv", a_log="A_log")
            mixer = PartSpec.of("channel_delta", hidden_size=H, num_heads=m.heads, num_kv_heads=m.kv_heads,
                                head_dim=m.dim, v_dim=m.vdim, conv=m.conv, eps=cfg.eps, unit_eps=UNIT_EPS,
                                tensor_prefix="mix.", tensor_names=names)
        else:
            a, b = m.left, m.right
            position = None
            if a.rot_dims:
                position = PartSpec.of("rotary", head_dim=a.dim, rotary_dim=a.rot_dims, theta=a.rot_base,
                                       interleaved=True, scaling={"kind": "linear", "factor": a.rot_factor})
            left = PartSpec.of("attention", hidden_size=H, num_heads=a.heads, num_kv_heads=a.kv_heads, head_dim=a.dim,
                               v_dim=a.vdim, window=a.window, scale=a.scale, position=position, qk_norm=cfg.eps,
                               qk_norm_span="row", sinks=True, gate="head", tensor_prefix="left.",
                               tensor_names={"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm",
                                             "k_norm": "k.norm", "sink": "sink", "g": "g"})
            right = PartSpec.of("state_space", hidden_size=H, num_heads=b.heads, v_dim=b.vdim, state=b.state,
                                groups=b.groups, conv=b.conv, norm_groups=b.norm_groups, eps=cfg.eps,
                                tensor_prefix="right.",
                                tensor_names={"in": "in", "conv": "conv", "conv_bias": "conv.b", "dt_bias": "dt_bias",
                                              "a_log": "A_log", "d": "D", "norm": "norm", "o": "o"})
            mixer = PartSpec.of("parallel", hidden_size=H, branches=(left, right), tensor_prefix="mix.",
                                scales=(m.left_scale, m.right_scale))
        ffn = None
        if L.ff is not None:
            ffn = PartSpec.of("gated_mlp", hidden_size=H, intermediate_size=L.ff, activation="silu",
                              tensor_prefix="mlp.", tensor_names={"gate": "gate", "up": "up", "down": "down"})
        layers.append(LayerSpec(block="post_norm", mixer=mixer, ffn=ffn,
                                norms=(_norm(H, cfg.eps, "norm1"), _norm(H, cfg.eps, "norm2")), prefix=f"l{i}.",
                                block_params=PartSpec.of("post_norm", hidden_size=H, multiplier=cfg.residual_mult)))
    return ModelSpec(
        hidden_size=H, vocab_size=cfg.vocab,
        embedding=PartSpec.of("token_embedding", vocab_size=cfg.vocab, hidden_size=H, name="embed"),
        layers=tuple(layers), order=tuple(Run(layer=i, cache=i) for i in range(len(layers))),
        final_norm=_norm(H, cfg.eps, "final.norm"),
        head=PartSpec.of("lm_head", vocab_size=cfg.vocab, hidden_size=H, name="lm_head", tied_to="embed"),
        max_positions=cfg.max_positions)


register_architecture("Biranex", BiranexConfig.from_json, biranex_spec)
