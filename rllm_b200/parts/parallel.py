"""``parallel``: two mixers side by side that read the same input; the result is
the mean of their outputs, each first divided by its root mean square over the
model width (eps inside the root) and multiplied by a weight of its own:

    y = 1/2 (rms(a(x)) * w_a + rms(b(x)) * w_b).

With ``scales`` = (c_a, c_b) the result is the weighted sum c_a a(x) + c_b b(x) instead, with
constants and no weights of its own; a block that can add the two in its next kernel takes them
unadded (``forward_terms``).  The branches' first products, where both give their weights away
(``Mixer.give_first_weight``), are then one product over the stacked weights.

Each branch is a registered mixer with its own ``PartSpec``, tensors (below its
``tensor_prefix``) and cache: the part's cache need is the branches' needs one
after the other (pages for one, state for the other, whatever they declare),
and each branch gets its own views.

params: hidden_size, eps, branches (two mixer ``PartSpec``s), tensor_names (key
"out": the two weights' names below the part's prefix, in branch order); or
hidden_size, branches, scales.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..kernels import ops
from .base import Mixer, StepContext, WeightedSum
from .linear import linear
from .registry import build_part, register_part
from .spec import PartSpec, TensorSpec


def _needs(mixer: Mixer) -> tuple:
    need = mixer.cache_need()
    if need is None:
        return ()
    return tuple(need) if isinstance(need, (tuple, list)) else (need,)


@register_part("mixer", "parallel")
class ParallelMixer(Mixer):
    def __init__(self, spec: PartSpec, prefix: str = ""):
        super().__init__(spec, prefix)
        p = spec.get()
        self.hidden = int(p["hidden_size"])
        scales = p.get("scales")
        self.scales = (float(scales[0]), float(scales[1])) if scales is not None else None
        self.eps = float(p["eps"]) if self.scales is None else 0.0
        branches = tuple(p["branches"])
        if len(branches) != 2:
            raise ValueError("a parallel mixer has two branches")
        self.branches: List[Mixer] = [
            build_part("mixer", b, prefix=prefix + str(b.get().get("tensor_prefix") or "")) for b in branches]
        names = dict(p.get("tensor_names") or ())
        out = tuple(names.get("out") or ())
        if self.scales is not None and out:
            raise ValueError("a parallel mixer with constant scales has no output weights")
        if self.scales is None and len(out) != 2:
            raise ValueError("a parallel spec names its two output weights: tensor_names with the key out")
        self.out_names = [prefix + str(n) for n in out]
        self.w_out: List[torch.Tensor] = []
        self.w_first: Optional[torch.Tensor] = None      # the branches' first weights, stacked
        self.first_rows: List[int] = []
        self.counts = [len(_needs(b)) for b in self.branches]
        self.several = [isinstance(b.cache_need(), (tuple, list)) for b in self.branches]

    @property
    def graph_safe(self) -> bool:
        return all(bool(b.graph_safe) for b in self.branches)

    def tensor_specs(self) -> List[TensorSpec]:
        specs = [ts for b in self.branches for ts in b.tensor_specs()]
        return specs + [TensorSpec(n, (self.hidden,), role="vector", init=("one_plus_normal", 0.1))
                        for n in self.out_names]

    def ignored_tensors(self) -> List[str]:
        return [n for b in self.branches for n in b.ignored_tensors()]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        for b in self.branches:
            b.load(tensors)
        self.w_first = None
        if self.scales is not None:
            self._stack_first()
            return
        self.w_out = [tensors[n].contiguous() for n in self.out_names]
        self.w_out[1] = self.w_out[1].to(self.w_out[0].dtype)

    def cache_need(self):
        return tuple(n for b in self.branches for n in _needs(b))

    def _stack_first(self) -> None:
        given = [b.give_first_weight() for b in self.branches]
        if any(w is None for w in given):
            for b, w in zip(self.branches, given):
                if w is not None:
                    b.take_back_first_weight(w)
            return
        rows, stack = [], []
        for w in given:
            rows.append(w.shape[0])
            stack.append(w)
            if w.shape[0] % 8:             # every branch's columns start on a 16-byte boundary in bfloat16
                stack.append(w.new_zeros((8 - w.shape[0] % 8, self.hidden)))
        self.first_rows = rows
        self.w_first = torch.cat(stack, dim=0).contiguous()

    def _outputs(self, x: torch.Tensor, ctx: StepContext, cache) -> List[torch.Tensor]:
        first = [None, None]
        if self.w_first is not None:
            a = linear(x, self.w_first)
            at = -(-self.first_rows[0] // 8) * 8
            first = [a[:, :self.first_rows[0]], a[:, at:at + self.first_rows[1]]]
        views = tuple(cache) if isinstance(cache, (tuple, list)) else ((cache,) if cache is not None else ())
        outs, at = [], 0
        for b, n, several, f in zip(self.branches, self.counts, self.several, first):
            mine = views[at:at + n]
            at += n
            extra = {} if f is None else {"first": f}
            outs.append(b.forward(x, ctx, mine if several else (mine[0] if n else None), **extra))
        return outs

    def forward_terms(self, x: torch.Tensor, ctx: StepContext, cache):
        """The two results and their factors, not added up; None: this mixer's result is no such sum."""
        if self.scales is None:
            return None
        return WeightedSum(tuple(self._outputs(x, ctx, cache)), self.scales)

    def forward(self, x: torch.Tensor, ctx: StepContext, cache) -> torch.Tensor:
        outs = self._outputs(x, ctx, cache)
        if self.scales is not None:
            return ops.scaled_sum2(outs[0], outs[1], *self.scales)
        return ops.rms_mean2(outs[0], outs[1], self.w_out[0], self.w_out[1], self.eps)
