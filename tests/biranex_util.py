"""Small Biranex configurations for the tests, none with a shipped model's sizes.

BX_A: sizes that are no multiples of 16 or 8.  A delta-rule layer whose heads share q/k heads (4 on 2, keys of 20,
values of 28, 3 taps) without a feed-forward; a parallel layer whose attention has keys of 24, values of 40, ten
rotated dims at a third of their frequency and a window of 11 (shorter than a page), beside a state-space part with
6 heads of 12 in 3 groups, 10 states, 2 taps and 4 norm groups; a delta-rule layer with as many q/k heads as heads,
9 taps and a feed-forward; a second parallel layer without a feed-forward, with a window over several pages.
BX_B: multiples of 16: the sizes of the tensor-core kernels (attention heads of 64 and 128 with keys and values of
one size, delta heads of 64 x 128 and 128 x 64, state-space heads of 64 x 64 and 128 x 32).
BX_C: a width that is no multiple of 8, and values that make mechanisms trivial: one head, one tap, a window of one token, nothing rotated but one pair and
no rescaling, a left scale of zero, a group a head; keys of 32 and values of 16 (rows of one size in the pages).
"""
from __future__ import annotations

import os


def delta(heads, kv, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}


def par(left, left_scale, right, right_scale):
    heads, kv, dim, vdim, scale, window, base, dims, factor = left
    rot = {"base": base, "dims": dims}
    if factor is not None:
        rot["scaling"] = {"factor": factor}
    sheads, svdim, state, groups, conv, norm_groups = right
    return {"left": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale,
                     "mask": {"size": window}, "rot": rot}, "left_scale": left_scale,
            "right": {"heads": sheads, "vdim": svdim, "state": state, "groups": groups, "conv": conv,
                      "norm_groups": norm_groups}, "right_scale": right_scale}


def layer(mixer, ff=None):
    return {"type": "parallel" if "left" in mixer else "channel_delta", "mixer": mixer,
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


BX_A = {
    "architecture": "Biranex", "vocab": 211, "width": 72, "norm": {"eps": 1e-5}, "residual_mult": 0.6,
    "layers": [
        layer(delta(4, 2, 20, 28, 3)),
        layer(par((6, 2, 24, 40, 0.3, 11, 300.0, 10, 3.0), 0.7, (6, 12, 10, 3, 2, 4), 0.9), 100),
        layer(delta(3, 3, 36, 12, 9), 60),
        layer(par((4, 1, 20, 20, 0.25, 53, 1000.0, 20, 5.0), 1.2, (4, 18, 33, 2, 5, 3), 0.4)),
    ],
}
BX_B = {
    "architecture": "Biranex", "vocab": 256, "width": 128, "norm": {"eps": 1e-6}, "residual_mult": 0.9,
    "layers": [
        layer(par((4, 4, 64, 64, 0.125, 64, 10000.0, 32, 4.0), 0.8, (2, 64, 64, 1, 4, 1), 0.7), 192),
        layer(delta(2, 2, 64, 128, 4), 64),
        layer(par((2, 1, 128, 128, 0.1, 33, 500.0, 128, 1.5), 0.5, (4, 32, 128, 2, 3, 2), 1.1)),
        layer(delta(2, 1, 128, 64, 2)),
    ],
}
BX_C = {
    "architecture": "Biranex", "vocab": 97, "width": 45, "norm": {"eps": 1e-3}, "residual_mult": 1.0,
    "layers": [
        layer(par((1, 1, 8, 12, 0.4, 1, 50.0, 2, None), 1.0, (1, 24, 1, 1, 1, 1), 1.0), 24),
        layer(delta(1, 1, 8, 4, 1)),
        layer(par((4, 2, 32, 16, 0.2, 19, 100.0, 32, 1.0), 0.0, (5, 8, 16, 5, 4, 5), 0.5), 16),
        layer(par((4, 2, 32, 16, 0.2, 19, 100.0, 16, 2.0), 1.0, (5, 8, 16, 5, 4, 1), 0.5)),
        layer(delta(2, 1, 33, 140, 3), 24),
    ],
}


def write_model(folder: str, cfg: dict, seed: int, edit=None) -> str:
    """A model folder with random weights; ``edit(weights dict)`` may change tensors before they are
    written (float32 storage)."""
    from rllm_b200.engine.loading import write_random_model
    write_random_model(folder, dict(cfg, torch_dtype="float32"), seed, "float32")
    if edit is not None:
        from safetensors import safe_open
        from safetensors.torch import save_file
        path = os.path.join(folder, "model.safetensors")
        with safe_open(path, framework="pt") as f:
            w = {n: f.get_tensor(n).clone() for n in f.keys()}
        edit(w)
        save_file({n: t.contiguous() for n, t in w.items()}, path)
    return folder


def sharpen(w: dict) -> None:
    """Make the mechanisms show: attention weights that differ (through the query norm's weight), gates and steps well away from
    nothing, half the decays slow, so that far tokens stay in the states, and the attention's branch as large as the
    one beside it (whose own norm makes it large whatever its input)."""
    for n, t in w.items():
        if n == "embed":
            t.mul_(20.0)
        elif n.endswith("left.v") or n.endswith("left.o"):
            t.mul_(5.0)
        elif n.endswith("left.q.norm"):
            t.mul_(1.5)
        elif n.endswith("left.g") or n.endswith("mix.b"):
            t.mul_(3.0)
        elif n.endswith("A_log"):
            t[::2] -= 3.0
        elif n.endswith("mix.a2"):
            t.mul_(2.0)


def other_ranks(w: dict) -> None:
    """The same, and the two low-rank pairs of every delta layer get ranks of their own: 5 and 19."""
    import torch
    sharpen(w)
    g = torch.Generator().manual_seed(5)
    for n in [n for n in w if n.endswith("mix.a1") or n.endswith("mix.g1")]:
        rank = 5 if n.endswith("a1") else 19
        second = n[:-1] + "2"
        w[n] = torch.randn(rank, w[n].shape[1], generator=g) * 0.2
        w[second] = torch.randn(w[second].shape[0], rank, generator=g) * 0.3
