"""A plain, slow Bikovik in float64, written from the design's equations: one
function per mechanism, whole sequences only, no cache, no batching.  It is what
the engine's Bikovik is compared with and shares no code with it.

Weights: a dict name -> float64 tensor.  Configuration: the dict of config.json.
"""
from __future__ import annotations

import json
import math
import os
from typing import Dict, List, Optional

import torch

F64 = torch.float64
GATE_SLOPE = 1.702


def read_model_dir(model_dir: str, round_to: Optional[torch.dtype] = None):
    """``round_to``: the matrices are rounded to it (vectors and head mixtures of a 32-bit file keep their digits)."""
    from safetensors import safe_open
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    w = {}
    with safe_open(os.path.join(model_dir, "model.safetensors"), framework="pt") as f:
        for n in f.keys():
            t = f.get_tensor(n)
            matrix = t.dim() == 2 and not n.endswith(".talk")
            w[n] = (t.to(round_to) if round_to is not None and matrix else t).to(F64)
    return cfg, w


# ---------------------------------------------------------------------------
# small functions
# ---------------------------------------------------------------------------
def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps)


def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * sigmoid(z)


def dynamic_tanh(w, name: str, x: torch.Tensor) -> torch.Tensor:
    return torch.tanh(w[name + ".alpha"] * x) * w[name] + w[name + ".b"]


def soft_cap(x: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(x / cap)


def rotate_halves(x: torch.Tensor, base: float, dims: int, positions: torch.Tensor) -> torch.Tensor:
    """x [T, heads, d]: dimensions i and i + dims / 2 turned by position * base^(-2i / dims); the rest as it is."""
    out, half = x.clone(), dims // 2
    for i in range(half):
        a = positions.to(F64)[:, None] * base ** (-2.0 * i / dims)
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., i + half] = v * torch.cos(a) + u * torch.sin(a)
    return out


def rotated(x: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    return x if rot is None else rotate_halves(x, float(rot["base"]), int(rot["dims"]), torch.arange(x.shape[0]))


# ---------------------------------------------------------------------------
# attention
# ---------------------------------------------------------------------------
def visible(T: int, window: Optional[int], keep: int) -> torch.Tensor:
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    return seen if window is None else seen & ((i - j < window) | (j < keep))


def talking_scores(q: torch.Tensor, k: torch.Tensor, scale: float, talk: torch.Tensor) -> torch.Tensor:
    """q [T, H, d], k [T, G, d] -> [H, T, T]: every head's scores, then the heads' mixture of them."""
    H, G = q.shape[1], k.shape[1]
    s = torch.stack([(q[:, h] @ k[:, h // (H // G)].t()) * scale for h in range(H)])
    return torch.einsum("hg,gij->hij", talk, s)


def attention(w, pre: str, m: dict, h: torch.Tensor, eps: float, shared: dict) -> torch.Tensor:
    T, H, G, d, dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q, k, v = (h @ w[pre + n].t() + w[pre + n + ".b"] for n in "qkv")
    q, k, v = rotated(q.view(T, H, d), m.get("rot")), rotated(k.view(T, G, d), m.get("rot")), v.view(T, G, dv)
    if m.get("v_mix"):
        if "v_first" in shared:
            lam = w[pre + "vmix"]
            v = (1.0 - lam) * v + lam * shared["v_first"]
        else:
            shared["v_first"] = v
    s = talking_scores(q, k, float(m["scale"]), w[pre + "talk"])
    mask = m.get("mask")
    seen = visible(T, int(mask["size"]), int(mask.get("keep_first", 0))) if mask else visible(T, None, 0)
    p = torch.softmax(s.masked_fill(~seen, -math.inf), dim=-1)
    o = torch.stack([p[hd] @ v[:, hd // (H // G)] for hd in range(H)], dim=1)
    return o.reshape(T, H * dv) @ w[pre + "o"].t()


# ---------------------------------------------------------------------------
# recurrences, token by token
# ---------------------------------------------------------------------------
def linear_state(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, keep: torch.Tensor) -> torch.Tensor:
    """S_t = diag(keep_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t.  q, k, keep [T, heads, d], v [T, heads, dv]."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=F64)
    o = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        S = keep[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return o


def forget_gate(z: torch.Tensor, lower: torch.Tensor) -> torch.Tensor:
    return lower + (1.0 - lower) * sigmoid(z)


def hgrn2(w, pre: str, m: dict, h: torch.Tensor, eps: float, shared: dict) -> torch.Tensor:
    T, H, d, dv = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q, v = silu(h @ w[pre + "q"].t()).view(T, H, d), (h @ w[pre + "v"].t()).view(T, H, dv)
    f = forget_gate(h @ w[pre + "f"].t() + w[pre + "f.b"], w[pre + "lower"]).view(T, H, d)
    o = rms(linear_state(q, 1.0 - f, v, f), eps) * w[pre + "norm"]
    return o.reshape(T, H * dv) @ w[pre + "o"].t()


def retention(w, pre: str, m: dict, h: torch.Tensor, eps: float, shared: dict) -> torch.Tensor:
    T, H, d, dv = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = rotated((h @ w[pre + "q"].t()).view(T, H, d), m.get("rot"))
    k = rotated((h @ w[pre + "k"].t()).view(T, H, d), m.get("rot")) * d ** -0.5
    v = (h @ w[pre + "v"].t()).view(T, H, dv)
    keep = torch.tensor([float(x) for x in m["decay"]], dtype=F64)[None, :, None].expand(T, H, d)
    o = rms(linear_state(q, k, v, keep), eps).reshape(T, H * dv)
    return (o * silu(h @ w[pre + "g"].t())) @ w[pre + "o"].t()


# ---------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------
def clamped_ff(w, pre: str, x: torch.Tensor, limit: float) -> torch.Tensor:
    g = torch.clamp(x @ w[pre + "gate"].t(), max=limit)
    u = torch.clamp(x @ w[pre + "up"].t(), min=-limit, max=limit)
    return (g * sigmoid(GATE_SLOPE * g) * (u + 1.0)) @ w[pre + "down"].t()


MIXERS = {"attention": attention, "hgrn2": hgrn2, "retention": retention}


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], collect: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence from position 0; ``collect`` gets the stream after every layer."""
    eps, shared = float(cfg["norm"]["eps"]), {}
    x = w["embed"][torch.tensor(tokens)] * float(cfg["embedding"]["scale"])
    for i, L in enumerate(cfg["layers"]):
        pre = f"l{i}."
        x = x + MIXERS[L["type"]](w, pre + "mix.", L["mixer"], dynamic_tanh(w, pre + "norm1", x), eps, shared)
        if L.get("mlp") is not None:
            x = x + clamped_ff(w, pre + "mlp.", dynamic_tanh(w, pre + "norm2", x), float(L["mlp"]["limit"]))
        if collect is not None:
            collect.append(x.clone())
    return soft_cap(dynamic_tanh(w, "final.norm", x) @ w["head"].t(), float(cfg["logit_softcap"]))
