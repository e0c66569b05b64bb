"""A plain, slow Biranex in float64, written from the design's equations: one
function per mechanism, whole sequences only, no cache, no batching.  It is what
the engine's Biranex is compared with and shares no code with it.

Weights: a dict name -> float64 tensor.  Configuration: the dict of config.json.
"""
from __future__ import annotations

import json
import math
import os
from typing import Dict, List, Optional

import torch

F64 = torch.float64
UNIT_EPS = 1e-6


def read_model_dir(model_dir: str, round_to: Optional[torch.dtype] = None):
    from safetensors import safe_open
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    w = {}
    with safe_open(os.path.join(model_dir, "model.safetensors"), framework="pt") as f:
        for n in f.keys():
            t = f.get_tensor(n)
            w[n] = (t.to(round_to) if round_to is not None and t.is_floating_point() else t).to(F64)
    return cfg, w


# ---------------------------------------------------------------------------
# small functions
# ---------------------------------------------------------------------------
def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z / (1.0 + torch.exp(-z))


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt(x.pow(2).sum(dim=-1, keepdim=True) + UNIT_EPS)


def short_conv(x: torch.Tensor, taps: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """x [T, C], taps [C, n]: y_t = sum_j taps[:, j] x_(t - (n - 1) + j), zeros ahead of the start."""
    T, n = x.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(n - 1, x.shape[1], dtype=x.dtype), x], dim=0)
    y = sum(taps[:, j] * padded[j:j + T] for j in range(n))
    return y if bias is None else y + bias


# ---------------------------------------------------------------------------
# positions
# ---------------------------------------------------------------------------
def rotation_frequencies(rot: dict) -> List[float]:
    dims, base = int(rot["dims"]), float(rot["base"])
    slow = float(rot["scaling"]["factor"]) if rot.get("scaling") else 1.0
    return [base ** (-2.0 * i / dims) / slow for i in range(dims // 2)]


def rotate_pairs(x: torch.Tensor, rot: dict, positions: torch.Tensor) -> torch.Tensor:
    """x [T, heads, d]: dimensions 2i and 2i + 1 turned by position * f_i; the rest as it is."""
    out = x.clone()
    for i, f in enumerate(rotation_frequencies(rot)):
        a = positions.to(F64)[:, None] * f
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., 2 * i + 1] = v * torch.cos(a) + u * torch.sin(a)
    return out


# ---------------------------------------------------------------------------
# mixers (h [T, width] of one sequence from position 0)
# ---------------------------------------------------------------------------
def window_attention(w, pre: str, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    T, H, G, d, dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    pos = torch.arange(T)
    q = rms(h @ w[pre + "q"].t(), eps) * w[pre + "q.norm"]            # one norm over all heads together
    k = rms(h @ w[pre + "k"].t(), eps) * w[pre + "k.norm"]
    q = rotate_pairs(q.view(T, H, d), m["rot"], pos)
    k = rotate_pairs(k.view(T, G, d), m["rot"], pos)
    v = (h @ w[pre + "v"].t()).view(T, G, dv)
    gate = torch.sigmoid(h @ w[pre + "g"].t())
    dist = pos[:, None] - pos[None, :]
    seen = (dist >= 0) & (dist < int(m["mask"]["size"]))
    outs = []
    for hd in range(H):
        g = hd // (H // G)
        s = ((q[:, hd] @ k[:, g].t()) * float(m["scale"])).masked_fill(~seen, -math.inf)
        sink = w[pre + "sink"][hd]
        top = torch.maximum(s.max(dim=-1, keepdim=True).values, sink)
        e = torch.exp(s - top)
        p = e / (torch.exp(sink - top) + e.sum(dim=-1, keepdim=True))
        outs.append((p @ v[:, g]) * gate[:, hd:hd + 1])
    return torch.cat(outs, dim=-1) @ w[pre + "o"].t()


def state_space(x: torch.Tensor, B: torch.Tensor, C: torch.Tensor, dt: torch.Tensor, rate: torch.Tensor,
                D: torch.Tensor) -> torch.Tensor:
    """Token by token.  x [T, heads, v], B, C [T, groups, n], dt [T, heads] (after softplus), rate [heads] > 0."""
    T, H, V = x.shape
    per = H // B.shape[1]
    S = torch.zeros(H, B.shape[2], V, dtype=F64)
    y = torch.zeros(T, H, V, dtype=F64)
    for t in range(T):
        for hd in range(H):
            g = hd // per
            S[hd] = torch.exp(-rate[hd] * dt[t, hd]) * S[hd] + dt[t, hd] * torch.outer(B[t, g], x[t, hd])
            y[t, hd] = C[t, g] @ S[hd] + D[hd] * x[t, hd]
    return y


def ssd(w, pre: str, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    T, H, dv, N, G = h.shape[0], int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"])
    inner = H * dv
    z, xbc, dt = torch.split(h @ w[pre + "in"].t(), [inner, inner + 2 * G * N, H], dim=-1)
    xbc = silu(short_conv(xbc, w[pre + "conv"], w[pre + "conv.b"]))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], dim=-1)
    y = state_space(x.reshape(T, H, dv), B.reshape(T, G, N), C.reshape(T, G, N), softplus(dt + w[pre + "dt_bias"]),
                    torch.exp(w[pre + "A_log"]), w[pre + "D"])
    y = y.reshape(T, inner) * silu(z)
    parts = int(m["norm_groups"])
    y = rms(y.view(T, parts, inner // parts), eps).reshape(T, inner) * w[pre + "norm"]
    return y @ w[pre + "o"].t()


def parallel(w, pre: str, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    return float(m["left_scale"]) * window_attention(w, pre + "left.", m["left"], h, eps) + \
        float(m["right_scale"]) * ssd(w, pre + "right.", m["right"], h, eps)


def delta_memory(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, g: torch.Tensor, beta: torch.Tensor) -> torch.Tensor:
    """Token by token.  q, k, g [T, heads, d] (g the decays), v [T, heads, dv], beta [T, heads]."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=F64)
    o = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return o


def channel_delta(w, pre: str, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    T, H, G, d, dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q, k, v = (silu(short_conv(h @ w[pre + n].t(), w[pre + n + ".conv"])) for n in "qkv")
    share = [hd // (H // G) for hd in range(H)]
    q = unit(q.view(T, G, d))[:, share] * d ** -0.5
    k = unit(k.view(T, G, d))[:, share]
    beta = torch.sigmoid(h @ w[pre + "b"].t())
    step = softplus((h @ w[pre + "a1"].t()) @ w[pre + "a2"].t() + w[pre + "dt_bias"]).view(T, H, d)
    g = torch.exp(-torch.exp(w[pre + "A_log"])[None, :, None] * step)
    o = delta_memory(q, k, v.view(T, H, dv), g, beta)
    gate = torch.sigmoid((h @ w[pre + "g1"].t()) @ w[pre + "g2"].t()).view(T, H, dv)
    return (rms(o, eps) * w[pre + "norm"] * gate).reshape(T, H * dv) @ w[pre + "o"].t()


def dense_ff(w, pre: str, x: torch.Tensor) -> torch.Tensor:
    return (silu(x @ w[pre + "gate"].t()) * (x @ w[pre + "up"].t())) @ w[pre + "down"].t()


# ---------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------
MIXERS = {"parallel": parallel, "channel_delta": channel_delta}


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], collect: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence from position 0; ``collect`` gets the stream after every layer."""
    eps, mult = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    x = w["embed"][torch.tensor(tokens)]
    for i, L in enumerate(cfg["layers"]):
        pre = f"l{i}."
        x = x + mult * rms(MIXERS[L["type"]](w, pre + "mix.", L["mixer"], x, eps), eps) * w[pre + "norm1"]
        if L.get("mlp") is not None:
            x = x + mult * rms(dense_ff(w, pre + "mlp.", x), eps) * w[pre + "norm2"]
        if collect is not None:
            collect.append(x.clone())
    return (rms(x, eps) * w["final.norm"]) @ w["embed"].t()
