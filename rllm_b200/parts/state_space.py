"""``state_space``: the Mamba-2 mixer (state-space duality form: one decay per head and token).

    [z | u | dt] = W_in h            z: inner = heads * v values, u: inner + 2 groups * state, dt: heads
    [x | B | C] = silu(conv_bias + sum_j conv[ch, j] u_{t - (taps - 1) + j})       (zeros before the start)
    dt <- softplus(dt + dt_bias)
    per head, with the B and C of its group:
        S_t = exp(-exp(a_log) dt_t) S_(t-1) + dt_t B_t x_t^T          [state, v]
        y_t = S_t^T C_t + d x_t
    y <- y * silu(z);   each of ``norm_groups`` equal parts of y over its own root mean square (eps inside
    the root), times the norm weight;   out = W_o y

Per request the part keeps two states, both float32: S [heads, state, v] and the convolution's last
taps - 1 inputs ([taps - 1, channels]); both start at zero.  The projections are matrix products in the
activation dtype (that of the steps dt keeps its float32 result); step sizes, decays, exponentials, the
state, the sums and the norm are float32 in the kernels.  Long portions are scanned as chunks side by side
(``ops.ssd_scan``).

params: hidden_size, num_heads, v_dim, state, groups, conv (taps), norm_groups, eps, tensor_names (keys
"in", "conv", "conv_bias", "dt_bias", "a_log", "d", "norm", "o").
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..kernels import ops
from .base import Mixer, StepContext
from .linear import linear
from .registry import register_part
from .spec import PartSpec, StateNeed, TensorSpec

_KEYS = ("in", "conv", "conv_bias", "dt_bias", "a_log", "d", "norm", "o")


@register_part("mixer", "state_space")
class StateSpace(Mixer):
    graph_safe = True

    def __init__(self, spec: PartSpec, prefix: str = ""):
        super().__init__(spec, prefix)
        p = spec.get()
        self.hidden, self.heads, self.dv = int(p["hidden_size"]), int(p["num_heads"]), int(p["v_dim"])
        self.state, self.groups, self.taps = int(p["state"]), int(p["groups"]), int(p["conv"])
        self.norm_groups, self.eps = int(p["norm_groups"]), float(p["eps"])
        self.inner = self.heads * self.dv
        self.channels = self.inner + 2 * self.groups * self.state
        if min(self.heads, self.dv, self.state, self.groups, self.taps, self.norm_groups) < 1:
            raise ValueError("state_space: sizes must be positive")
        if self.heads % self.groups or self.inner % self.norm_groups:
            raise ValueError("state_space: heads in whole groups, channels in whole norm groups")
        if self.state > 256:
            raise ValueError(f"state_space: state {self.state}; the scan kernels take up to 256")
        names = dict(p.get("tensor_names") or ())
        if sorted(names) != sorted(_KEYS):
            raise ValueError(f"a state_space spec names its tensors: tensor_names with the keys {_KEYS}")
        self.names = {k: prefix + str(v) for k, v in names.items()}
        self.w_in: Optional[torch.Tensor] = None
        self.w: Dict[str, torch.Tensor] = {}

    def tensor_specs(self) -> List[TensorSpec]:
        n, H, C = self.names, self.hidden, self.channels
        return [TensorSpec(n["in"], (self.inner + C + self.heads, H)),
                TensorSpec(n["conv"], (C, self.taps), role="vector", init=("normal", 0.4)),
                TensorSpec(n["conv_bias"], (C,), role="vector", init=("normal", 0.1)),
                TensorSpec(n["dt_bias"], (self.heads,), role="vector", init=("normal", 1.0)),
                TensorSpec(n["a_log"], (self.heads,), role="vector", init=("normal", 1.0)),
                TensorSpec(n["d"], (self.heads,), role="vector", init=("one_plus_normal", 0.1)),
                TensorSpec(n["norm"], (self.inner,), role="vector", init=("one_plus_normal", 0.1)),
                TensorSpec(n["o"], (H, self.inner))]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        n = self.names
        w_in = tensors[n["in"]]
        rows = self.inner + self.channels
        self.w_in = w_in[:rows].contiguous()
        self.w = {"dt": w_in[rows:].contiguous(), "o": tensors[n["o"]], "conv": tensors[n["conv"]].contiguous()}
        self.w["conv_bias"] = tensors[n["conv_bias"]].to(self.w["conv"].dtype).contiguous()
        # a few numbers per head and channel that enter float32 arithmetic: kept so
        for k in ("dt_bias", "a_log", "d", "norm"):
            self.w[k] = tensors[n[k]].float().contiguous()

    def cache_need(self):
        return (StateNeed((self.heads, self.state, self.dv)), StateNeed((self.taps - 1, self.channels)))

    def give_first_weight(self) -> Optional[torch.Tensor]:
        w, self.w_in = self.w_in, None
        return w

    def take_back_first_weight(self, weight: torch.Tensor) -> None:
        self.w_in = weight

    def forward(self, x: torch.Tensor, ctx: StepContext, cache, first: Optional[torch.Tensor] = None) -> torch.Tensor:
        scan_state, tail = cache
        w, E = self.w, self.inner
        a = linear(x, self.w_in) if first is None else first               # [T, inner + channels]: z | u
        dt = linear(x, w["dt"], out_dtype=torch.float32)                   # [T, heads]
        c = ops.causal_conv(a[:, E:], w["conv"], w["conv_bias"], tail.state, ctx.q_start, ctx.token_seq,
                            ctx.state_slots, ctx.num_seqs, ctx.num_tokens > ctx.num_decode, ctx.err)
        y = ops.ssd_scan(c, dt, w["dt_bias"], w["a_log"], w["d"], scan_state.state, ctx.q_start, ctx.state_slots,
                         ctx.num_seqs, self.heads, self.groups, self.state, self.dv, ctx.err,
                         max_q_len=ctx.max_q_len)                          # float32 [T, inner]
        y = ops.silu_gated_group_rmsnorm(y, a[:, :E], w["norm"], self.eps, self.norm_groups, x.dtype)
        return linear(y, w["o"])
