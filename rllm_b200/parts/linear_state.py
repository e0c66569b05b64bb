"""Linear attention with a matrix state a head, S_t = diag(f_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, in two kinds:

``retention``   fixed decays and rotated queries and keys
    q = W_q h, k = W_k h  [heads, head_dim],   v = W_v h  [heads, v_dim]
    q, k rotated by position, then k multiplied by head_dim^(-1/2);   f = decay[head]
    y = W_o ([o over its root mean square, per head] * silu(W_g h))
``hgrn2``       a decay per head and key channel, one minus which is the key
    q = silu(W_q h), v = W_v h,   f = l + (1 - l) sigmoid(W_f h + b),   k = 1 - f
    y = W_o [o over its root mean square, times w [v_dim], per head]

(eps inside the roots.)  S is float32 [heads, head_dim, v_dim] per request, starts at zero and is carried from step to
step in the request's state slot.  The input projections are one matrix product over the stacked weights in the
activation dtype; everything from there to y's last product is float32 arithmetic in one kernel call
(``ops.linear_state_scan``).

params: hidden_size, num_heads, head_dim, v_dim, eps, tensor_names; retention also decay (one number a head) and
position (PartSpec of a rotation of halves, or None); tensor_names have the keys q, k, v, g, o (retention) or q, f,
f_bias, lower, v, norm, o (hgrn2).
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..kernels import ops
from .base import Mixer, StateCacheView, StepContext
from .linear import fused_residual_takes, linear
from .registry import build_part, register_part
from .spec import PartSpec, StateNeed, TensorSpec


class LinearStateMixer(Mixer):
    graph_safe = True
    keys = ()                     # tensor_names of the kind
    stacked = ()                  # its input projections, in the order of the product's columns

    def __init__(self, spec: PartSpec, prefix: str = ""):
        super().__init__(spec, prefix)
        p = spec.get()
        self.hidden, self.heads = int(p["hidden_size"]), int(p["num_heads"])
        self.d, self.dv, self.eps = int(p["head_dim"]), int(p["v_dim"]), float(p["eps"])
        if self.d > 512 or (self.dv % 4 and self.d > 256):
            raise ValueError(f"{spec.kind}: head_dim {self.d}; the scan kernels take up to 512 (256 where v_dim is no "
                             "multiple of 4)")
        names = dict(p.get("tensor_names") or ())
        if sorted(names) != sorted(self.keys):
            raise ValueError(f"a {spec.kind} spec names its tensors: tensor_names with the keys {sorted(self.keys)}")
        self.names = {k: prefix + str(v) for k, v in names.items()}
        self.w_in: Optional[torch.Tensor] = None
        self.w_o: Optional[torch.Tensor] = None

    def _rows(self, key: str) -> int:
        return self.heads * (self.dv if key in ("v", "g") else self.d)

    def tensor_specs(self) -> List[TensorSpec]:
        n = self.names
        return [TensorSpec(n[k], (self._rows(k), self.hidden)) for k in self.stacked] + \
            [TensorSpec(n["o"], (self.hidden, self.heads * self.dv))]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.w_in = torch.cat([tensors[self.names[k]] for k in self.stacked], dim=0).contiguous()
        self.w_o = tensors[self.names["o"]]

    def cache_need(self):
        return StateNeed((self.heads, self.d, self.dv))

    def fused_residual(self, num_rows: int, dtype: torch.dtype) -> bool:
        return fused_residual_takes(num_rows, dtype, self.w_in, self.w_o)

    def _scan(self, a: torch.Tensor, ctx: StepContext, **kind) -> torch.Tensor:
        """``kind``: the arguments of ``ops.linear_state_scan`` that this kind of recurrence needs."""
        return ops.linear_state_scan(a, kind.pop("state"), ctx.q_start, ctx.state_slots, ctx.num_seqs, self.eps, ctx.err,
                                     positions=ctx.positions, max_q_len=ctx.max_q_len, early=True,
                                     num_decode=ctx.num_decode, tables=ctx.extras.setdefault("tables", {}), **kind)

    def recurrence(self, a: torch.Tensor, ctx: StepContext, state: torch.Tensor) -> torch.Tensor:
        """From the tokens' projections to the output product's input."""
        raise NotImplementedError

    def forward(self, x, ctx: StepContext, cache: StateCacheView, residual=None):
        y = self.recurrence(linear(x, self.w_in), ctx, cache.state)
        return linear(y, self.w_o, residual=residual)


@register_part("mixer", "retention")
class Retention(LinearStateMixer):
    keys = ("q", "k", "v", "g", "o")
    stacked = ("q", "k", "v", "g")

    def __init__(self, spec: PartSpec, prefix: str = ""):
        super().__init__(spec, prefix)
        p = spec.get()
        self.decay = tuple(float(v) for v in p["decay"])
        if len(self.decay) != self.heads:
            raise ValueError(f"retention: {len(self.decay)} decays for {self.heads} heads")
        pos = p.get("position")
        self.position = build_part("position_encoding", pos if pos is not None else PartSpec.of("none"), prefix=prefix)
        if self.position.fused_rotary() is None or getattr(self.position, "interleaved", False) or \
                float(getattr(self.position, "magnitude", 1.0)) != 1.0:
            raise ValueError("retention takes a plain rotation of halves, or none")
        self.decay_dev: Optional[torch.Tensor] = None

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        super().load(tensors)
        self.decay_dev = torch.tensor(self.decay, dtype=torch.float32, device=self.w_o.device)

    def recurrence(self, a, ctx, state):
        inv_freq, rd = self.position.fused_rotary(a.device)
        return self._scan(a, ctx, state=state, decay=self.decay_dev, inv_freq=inv_freq, rotary_dim=rd,
                          k_scale=float(self.d) ** -0.5, gated=True)


@register_part("mixer", "hgrn2")
class Hgrn2(LinearStateMixer):
    keys = ("q", "f", "f_bias", "lower", "v", "norm", "o")
    stacked = ("q", "f", "v")

    def __init__(self, spec: PartSpec, prefix: str = ""):
        super().__init__(spec, prefix)
        self.f_bias = self.lower = self.norm = None

    def tensor_specs(self) -> List[TensorSpec]:
        n, ch = self.names, self.heads * self.d
        return super().tensor_specs() + [
            TensorSpec(n["f_bias"], (ch,), role="vector", init=("normal", 1.0)),
            TensorSpec(n["lower"], (ch,), role="vector", init=("zeros",)),
            TensorSpec(n["norm"], (self.dv,), role="vector", init=("one_plus_normal", 0.1))]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        super().load(tensors)
        # a few numbers per channel that enter float32 arithmetic: kept so
        self.f_bias, self.lower, self.norm = (tensors[self.names[k]].float().contiguous()
                                              for k in ("f_bias", "lower", "norm"))

    def recurrence(self, a, ctx, state):
        return self._scan(a, ctx, state=state, f_bias=self.f_bias, lower=self.lower, norm=self.norm)
