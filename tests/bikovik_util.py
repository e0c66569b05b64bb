"""Small Bikovik configurations for the tests, none with a shipped model's sizes.

BK_A: sizes that are no multiples of 16 or 8, all three kinds and a layer without a feed-forward: HGRN2 with heads of
20 x 28; attention with 6 heads on 2, keys of 20, values of 12, a window of 11 (shorter than a page) beside 3 kept tokens
and mixed values; retention with heads of 24 x 40 that rotate in part; attention without mixed values (two heads on two,
keys of 36, nothing kept, a window over several pages); attention with the first one's kv heads and values, mixed.
BK_B: multiples of 16, sizes of the tensor-core kernels: attention with 8 heads on 2, keys of 64 and values of 32 (and 4 on
4 with keys of 128: a key row of eight panels), HGRN2 with heads of 64 x 128, retention with heads of 128 x 64.
BK_C: a width that is no multiple of 8, and values that make mechanisms trivial: one head, a window of one token, more kept
tokens than the window, a layer that sees every key, nothing rotated, a decay of zero and one of one, an embedding scale of
one, a gate that the clamp hardly reaches.
"""
from __future__ import annotations

import os


def att(heads, kv, dim, vdim, scale, window, keep, base, dims, v_mix, ff=None, limit=2.0):
    mixer = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if dims:
        mixer["rot"] = {"base": base, "dims": dims}
    if window is not None:
        mixer["mask"] = {"size": window, "keep_first": keep}
    return _layer("attention", mixer, ff, limit)


def hgrn2(heads, dim, vdim, ff=None, limit=2.0):
    return _layer("hgrn2", {"heads": heads, "dim": dim, "vdim": vdim}, ff, limit)


def ret(heads, dim, vdim, decay, base, dims, ff=None, limit=2.0):
    mixer = {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}
    if dims:
        mixer["rot"] = {"base": base, "dims": dims}
    return _layer("retention", mixer, ff, limit)


def _layer(kind, mixer, ff, limit):
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


BK_A = {
    "architecture": "Bikovik", "vocab": 211, "width": 72, "norm": {"eps": 1e-5}, "embedding": {"scale": 0.7},
    "logit_softcap": 11.0,
    "layers": [
        hgrn2(3, 20, 28, 100, 0.9),
        att(6, 2, 20, 12, 0.3, 11, 3, 300.0, 10, True, 60, 1.1),
        ret(2, 24, 40, [0.9, 0.997], 700.0, 16),
        att(2, 2, 36, 20, 0.2, 53, 0, 1000.0, 36, False, 44, 3.0),
        att(4, 2, 28, 12, 0.25, 30, 2, 200.0, 6, True),
    ],
}
BK_B = {
    "architecture": "Bikovik", "vocab": 256, "width": 128, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.5},
    "logit_softcap": 20.0,
    "layers": [
        att(8, 2, 64, 32, 0.125, 64, 5, 10000.0, 32, True, 192),
        hgrn2(2, 64, 128, 96),
        att(4, 2, 32, 32, 0.2, 33, 1, 500.0, 32, True, 64, 0.5),
        ret(2, 128, 64, [0.95, 0.998], 2000.0, 128, 128),
        att(4, 4, 128, 128, 0.09, 150, 20, 10000.0, 64, False, 160),
    ],
}
BK_C = {
    "architecture": "Bikovik", "vocab": 97, "width": 45, "norm": {"eps": 1e-3}, "embedding": {"scale": 1.0},
    "logit_softcap": 500.0,
    "layers": [
        att(1, 1, 8, 12, 0.4, 1, 0, 50.0, 2, True, 24, 100.0),
        ret(2, 10, 6, [0.0, 1.0], 1.0, 0, 16),
        att(5, 1, 9, 12, 0.3, 2, 7, 50.0, 8, True),
        hgrn2(1, 7, 5, 20, 0.01),
        att(2, 1, 16, 8, 0.2, None, 0, 1.0, 0, False, 16),
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
    """Make the mechanisms show: attention weights that differ, biases and head mixtures well away from nothing, gates
    that reach the clamp, forget gates with lower bounds and half of them slow, so that far tokens stay in the states."""
    import torch
    g = torch.Generator().manual_seed(3)
    for n in sorted(w):
        t = w[n]
        if n == "embed":
            t.mul_(30.0)
        elif n.endswith(("mix.q", "mix.k", "mix.g", "mlp.gate", "mlp.up")):
            t.mul_(8.0)
        elif n.endswith(("mix.v", "mix.o", "mlp.down")):
            t.mul_(4.0)
        elif n == "head":
            t.mul_(30.0)
        elif n.endswith(".talk"):
            t.add_(torch.eye(t.shape[0]))
        elif n.endswith(".lower"):
            t.copy_(torch.rand(t.shape, generator=g) * 0.9)
            t[::3] = 0.0
        elif n.endswith(".f.b"):
            t.mul_(2.0)
            t[::2] += 5.0
