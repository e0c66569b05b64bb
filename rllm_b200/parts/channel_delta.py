"""``channel_delta``: the gated delta rule with a decay of its own for every key channel.

    q = W_q h, k = W_k h  [kv_heads, d],   v = W_v h  [heads, dv];   each: a short causal convolution per
        channel (no bias, zeros before the start), then silu;   head h uses q/k head h // (heads / kv_heads)
    q <- q / sqrt(sum q^2 + unit_eps) * d^(-1/2),   k <- k / sqrt(sum k^2 + unit_eps)            (per head)
    beta = sigmoid(W_b h)  [heads];   g = exp(-exp(a_log_head) softplus(W_a2 (W_a1 h) + dt_bias))  [heads, d]
    S' = diag(g_t) S_(t-1);   u_t = beta_t (v_t - S'^T k_t);   S_t = S' + k_t u_t^T  [d, dv];   o_t = S_t^T q_t
    y = W_o (rms_per_head(o) * w * sigmoid(W_g2 (W_g1 h)))          (eps inside the root; w [dv] for all heads)

Per request the part keeps two states, both float32: S [heads, d, dv] and the convolutions' last taps - 1
inputs ([taps - 1, 2 kv_heads d + heads dv]); both start at zero.  q, k, v and the low-rank inputs W_a1 h,
W_g1 h are one matrix product over the stacked weights; beta's and the decays' pre-activations are products
whose results stay float32; unit vectors, logarithms, exponentials, the recurrence and the norm are float32
arithmetic in the kernels.  Steps in which every sequence brings one token take one kernel between the first
and the last product (``ops.channel_delta_step``).  The ranks of the two low-rank pairs are the tensors' own.

params: hidden_size, num_heads, num_kv_heads, head_dim, v_dim, conv (taps), eps, unit_eps, rank (optional: what
the random-weights mode draws; head_dim if absent), tensor_names (keys "q", "k", "v", "q_conv", "k_conv",
"v_conv", "b", "a1", "a2", "a_log", "dt_bias", "norm", "g1", "g2", "o").
"""
from __future__ import annotations

import os
from typing import Dict, List

import torch

from ..kernels import ops
from .base import Mixer, StepContext
from .linear import linear
from .registry import register_part
from .spec import FreeDim, PartSpec, StateNeed, TensorSpec

_KEYS = ("q", "k", "v", "q_conv", "k_conv", "v_conv", "b", "a1", "a2", "a_log", "dt_bias", "norm", "g1", "g2", "o")


def _rows8(w: torch.Tensor) -> torch.Tensor:
    """The weight with rows of zeros up to a multiple of 8 (its columns of a product then end on a 16-byte
    boundary in bfloat16)."""
    pad = -w.shape[0] % 8
    return w if not pad else torch.cat([w, w.new_zeros((pad, w.shape[1]))], dim=0)


def _cols8(w: torch.Tensor) -> torch.Tensor:
    pad = -w.shape[1] % 8
    return w.contiguous() if not pad else torch.cat([w, w.new_zeros((w.shape[0], pad))], dim=1).contiguous()


@register_part("mixer", "channel_delta")
class ChannelDelta(Mixer):
    graph_safe = True

    def __init__(self, spec: PartSpec, prefix: str = ""):
        super().__init__(spec, prefix)
        p = spec.get()
        self.hidden, self.heads, self.kv = int(p["hidden_size"]), int(p["num_heads"]), int(p["num_kv_heads"])
        self.d, self.dv, self.taps = int(p["head_dim"]), int(p["v_dim"]), int(p["conv"])
        self.eps, self.unit_eps = float(p["eps"]), float(p["unit_eps"])
        self.rank = int(p.get("rank") or self.d)
        if min(self.heads, self.kv, self.d, self.dv, self.taps) < 1 or self.heads % self.kv:
            raise ValueError("channel_delta: sizes must be positive, heads a multiple of kv_heads")
        if self.d > 256:
            raise ValueError(f"channel_delta: head_dim {self.d}; the scan kernels take up to 256")
        names = dict(p.get("tensor_names") or ())
        if sorted(names) != sorted(_KEYS):
            raise ValueError(f"a channel_delta spec names its tensors: tensor_names with the keys {_KEYS}")
        self.names = {k: prefix + str(v) for k, v in names.items()}
        self.qk, self.vv = self.kv * self.d, self.heads * self.dv
        self.channels = 2 * self.qk + self.vv
        self.w: Dict[str, torch.Tensor] = {}

    def tensor_specs(self) -> List[TensorSpec]:
        n, H, qk, vv = self.names, self.hidden, self.qk, self.vv
        ra, rg = FreeDim(self.rank, n["a1"]), FreeDim(self.rank, n["g1"])
        conv = dict(role="vector", init=("normal", 0.5))
        return [TensorSpec(n["q"], (qk, H)), TensorSpec(n["k"], (qk, H)), TensorSpec(n["v"], (vv, H)),
                TensorSpec(n["q_conv"], (qk, self.taps), **conv), TensorSpec(n["k_conv"], (qk, self.taps), **conv),
                TensorSpec(n["v_conv"], (vv, self.taps), **conv),
                TensorSpec(n["b"], (self.heads, H), init=("normal", 0.1)),
                TensorSpec(n["a1"], (ra, H)), TensorSpec(n["a2"], (self.heads * self.d, ra), init=("normal", 0.2)),
                TensorSpec(n["a_log"], (self.heads,), role="vector", init=("normal", 1.0)),
                TensorSpec(n["dt_bias"], (self.heads * self.d,), role="vector", init=("normal", 1.0)),
                TensorSpec(n["norm"], (self.dv,), role="vector", init=("one_plus_normal", 0.1)),
                TensorSpec(n["g1"], (rg, H)), TensorSpec(n["g2"], (vv, rg), init=("normal", 0.2)),
                TensorSpec(n["o"], (H, vv))]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        t = {k: tensors[n] for k, n in self.names.items()}
        qkv = _rows8(torch.cat([t["q"], t["k"], t["v"]], dim=0))
        a1, g1 = _rows8(t["a1"]), _rows8(t["g1"])
        self.at_a, self.at_g = qkv.shape[0], qkv.shape[0] + a1.shape[0]
        self.end_g = self.at_g + g1.shape[0]
        conv = torch.cat([t[k + "_conv"].to(t["q_conv"].dtype) for k in "qkv"], dim=0)
        self.w = {"in": torch.cat([qkv, a1, g1], dim=0).contiguous(), "conv": conv.contiguous(), "b": t["b"],
                  "a2": _cols8(t["a2"]), "g2": _cols8(t["g2"]), "o": t["o"],
                  # what enters float32 arithmetic is kept so, whatever the run's dtype
                  "a_log": t["a_log"].float().contiguous(), "dt_bias": t["dt_bias"].float().contiguous(),
                  "norm": t["norm"].float().repeat(self.heads).contiguous()}
        self.step_kernel = t["o"].is_cuda and os.environ.get("RLLM_CHANNEL_DELTA") != "simt" and \
            ops.channel_delta_step_takes(self.d, self.dv, self.w["a2"].shape[1], self.w["g2"].shape[1])

    def cache_need(self):
        return (StateNeed((self.heads, self.d, self.dv)), StateNeed((self.taps - 1, self.channels)))

    def _conv(self, a: torch.Tensor, tail, ctx: StepContext) -> torch.Tensor:
        return ops.causal_conv(a[:, :self.channels], self.w["conv"], None, tail.state, ctx.q_start, ctx.token_seq,
                               ctx.state_slots, ctx.num_seqs, ctx.num_tokens > ctx.num_decode, ctx.err)

    def forward(self, x: torch.Tensor, ctx: StepContext, cache) -> torch.Tensor:
        memory, tail = cache
        w = self.w
        a = linear(x, w["in"])                                               # q | k | v | W_a1 h | W_g1 h
        if ctx.num_tokens == ctx.num_decode and self.step_kernel:
            # decoding: everything up to the output product in one kernel (the convolutions too, unless heads
            # share a q/k head, whose last inputs then have one writer: the convolution's own kernel)
            c = None if self.kv == self.heads else self._conv(a, tail, ctx)
            y = ops.channel_delta_step(a, c, x, w, self.at_a, self.at_g, self.taps, self.unit_eps, self.eps,
                                       tail.state, memory.state, ctx.state_slots, self.heads, self.kv, self.d, self.dv,
                                       ctx.err, early=True)
            return linear(y, w["o"])
        b = linear(x, w["b"], out_dtype=torch.float32)                       # [T, heads]
        c = self._conv(a, tail, ctx)
        step = linear(a[:, self.at_a:self.at_g], w["a2"], out_dtype=torch.float32)     # [T, heads d]
        gate = linear(a[:, self.at_g:self.end_g], w["g2"])                             # [T, heads dv]
        o = ops.channel_delta_scan(c, step, b, w["dt_bias"], w["a_log"], self.unit_eps, memory.state, ctx.q_start,
                                   ctx.state_slots, ctx.num_seqs, self.heads, self.kv, self.d, self.dv, ctx.err,
                                   max_q_len=ctx.max_q_len)
        y = ops.head_gated_rmsnorm(o, gate, w["norm"], self.eps, self.heads, x.dtype)
        return linear(y, w["o"])
