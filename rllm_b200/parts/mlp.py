"""SiLU-gated feed-forward: down(silu(gate(x)) * up(x)), no bias
(crates/rllm-model/src/layers.rs:214-220).  gate and up are one matrix product
over the stacked weights [Wgate; Wup]; silu(z) = z / (1 + exp(-z)) and the
product with up are computed in float32.

``activation`` "gelu_tanh" puts 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3)))
in the place of the SiLU (one product over the stacked weights, then one kernel
for the activation and the product with up).

With the SiLU, ``limit``, ``slope`` and ``up_shift`` give the gate other constants: with g = min(gate(x), limit) and
u = up(x) kept within +-limit, down(g sigmoid(slope g) (u + up_shift)) (absent: no limit, 1, 0).

params: hidden_size, intermediate_size, activation ("silu" if absent), limit, slope, up_shift,
tensor_names (the names of the three weights below the part's prefix, keys
"gate", "up", "down").
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..kernels import ops
from .base import FeedForward
from .base import ScaledRows
from .linear import fused_residual_takes, linear
from .registry import register_part
from .spec import PartSpec, TensorSpec


@register_part("feed_forward", "gated_mlp")
class GatedMLP(FeedForward):
    graph_safe = True

    def __init__(self, spec: PartSpec, prefix: str = ""):
        super().__init__(spec, prefix)
        self.hidden = int(spec["hidden_size"])
        self.inter = int(spec["intermediate_size"])
        self.activation = str(spec.get().get("activation") or "silu")
        if self.activation not in ops.ACTIVATIONS:
            raise ValueError(f"activation {self.activation!r}; known: {sorted(ops.ACTIVATIONS)}")
        p = spec.get()
        self.gate = (float(p["limit"]) if p.get("limit") is not None else float("inf"),
                     float(p["slope"]) if p.get("slope") is not None else 1.0,
                     float(p["up_shift"]) if p.get("up_shift") is not None else 0.0)
        if self.gate != ops.PLAIN_GATE and self.activation != "silu":
            raise ValueError("limit, slope and up_shift go with the activation 'silu'")
        if not self.gate[0] > 0:
            raise ValueError("limit must be positive")
        names = dict(spec.get().get("tensor_names") or ())
        if sorted(names) != ["down", "gate", "up"]:
            raise ValueError("a gated_mlp spec names its weights: tensor_names with the keys gate, up, down")
        self.names = {k: str(v) for k, v in names.items()}
        self.w_gate_up: Optional[torch.Tensor] = None
        self.w_down: Optional[torch.Tensor] = None

    def _names(self):
        p = self.prefix
        return tuple(p + self.names[k] for k in ("gate", "up", "down"))

    def tensor_specs(self) -> List[TensorSpec]:
        g, u, d = self._names()
        return [TensorSpec(g, (self.inter, self.hidden)), TensorSpec(u, (self.inter, self.hidden)),
                TensorSpec(d, (self.hidden, self.inter))]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        g, u, d = self._names()
        self.w_gate_up = torch.cat([tensors[g], tensors[u]], dim=0).contiguous()
        self.w_down = tensors[d]

    def fused_residual(self, num_rows: int, dtype: torch.dtype) -> bool:
        return self.activation == "silu" and fused_residual_takes(num_rows, dtype, self.w_gate_up, self.w_down)

    def forward(self, x, residual=None):
        act = torch.empty((x.shape[0], self.inter), dtype=x.dtype, device=x.device)
        if self.activation != "silu":
            ops.act_mul(linear(x, self.w_gate_up), act, self.activation)
        elif isinstance(x, ScaledRows):
            # the rows' 1 / rms is applied to gate and up before the SiLU
            ops.gemm_small_m_rstd(x.x, x.parts, x.eps, self.w_gate_up, act, "silu_mul", gate=self.gate)
        elif ops.small_m_takes(x, self.w_gate_up):
            # few rows: one kernel streams [Wgate; Wup] once and applies silu(gate) * up to its accumulators
            ops.gemm_small_m(x, self.w_gate_up, act, "silu_mul", gate=self.gate)
        elif ops.tcgen05_takes(x, self.w_gate_up, silu=True):
            # many rows: tensor-core tiles of 128 gate and 128 up features, silu(gate) * up in the epilogue
            ops.gemm_tcgen05(x, self.w_gate_up, act, "silu_mul", gate=self.gate)
        else:
            gate_up = linear(x, self.w_gate_up)                   # [T, 2I]
            ops.silu_mul(gate_up, act, gate=self.gate)
        return linear(act, self.w_down, residual=residual)


@register_part("feed_forward", "plain_mlp")
class PlainMLP(FeedForward):
    """down(act(up(x))): two matrices, no gate and no bias; the activation is float32 arithmetic on the
    first product's result.

    params: hidden_size, intermediate_size, activation ("relu_squared": max(z, 0)^2, "silu", "gelu_tanh"),
    tensor_names (keys "up", "down")."""
    graph_safe = True

    def __init__(self, spec: PartSpec, prefix: str = ""):
        super().__init__(spec, prefix)
        self.hidden = int(spec["hidden_size"])
        self.inter = int(spec["intermediate_size"])
        self.activation = str(spec["activation"])
        if self.activation not in ops.PLAIN_ACTIVATIONS:
            raise ValueError(f"activation {self.activation!r}; known: {sorted(ops.PLAIN_ACTIVATIONS)}")
        names = dict(spec.get().get("tensor_names") or ())
        if sorted(names) != ["down", "up"]:
            raise ValueError("a plain_mlp spec names its weights: tensor_names with the keys up, down")
        self.names = {k: prefix + str(v) for k, v in names.items()}
        self.w_up: Optional[torch.Tensor] = None
        self.w_down: Optional[torch.Tensor] = None

    def tensor_specs(self) -> List[TensorSpec]:
        return [TensorSpec(self.names["up"], (self.inter, self.hidden)),
                TensorSpec(self.names["down"], (self.hidden, self.inter))]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.w_up, self.w_down = tensors[self.names["up"]], tensors[self.names["down"]]

    def forward(self, x):
        u = linear(x, self.w_up)
        ops.act(u, u, self.activation)
        return linear(u, self.w_down)
