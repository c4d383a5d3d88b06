"""Two mixers side by side on the same input:  out = left(x1) + right(x1), each with its own multiplier (``out_scale`` of
the mixer).

Both leave what their output products read (``Mixer.forward_rows``) in the halves of one row, and ONE product with both
output matrices side by side, [Wo_left | Wo_right], adds the two: no sum of its own, one rounding.  Where both begin with
a product of x1 (``Mixer.in_weight``), ONE product does both, weight "win".  Parameters carry the
prefix "left." or "right."; the bound output weight is "wo".  One of the two may keep a cache, one may carry state.
"""
from __future__ import annotations

import torch

from .base import MIXERS, Mixer
from .linear import matmul_nt, stack_products


@MIXERS.register("side_by_side")
class SideBySide(Mixer):
    """params: width, left, right (PartSpecs of mixers that leave rows)."""

    def __init__(self, params, dtype, device):
        super().__init__(params, dtype, device)
        self.d = int(params["width"])
        self.sides = {n: MIXERS.build(params[n], dtype, device) for n in ("left", "right")}
        for n, m in self.sides.items():
            if m.rows_width is None:
                raise ValueError(f"a mixer of kind {params[n].kind!r} does not leave its rows to another part's product")
        self.tile_sizes = sorted({int(t) for m in self.sides.values() for t in getattr(m, "tile_sizes", ())})
        biased = [n for n, m in self.sides.items() if m.has_out_bias]
        if len(biased) > 1:
            raise ValueError("only one of two mixers side by side may have a bias on its output")
        self.has_out_bias = bool(biased)
        if all(m.in_weight for m in self.sides.values()):
            self.in_weight = "win"
        self.cached = self._the_one("cache", lambda m: m.cache_need())
        self.stateful = self._the_one("state", lambda m: m.state_need())

    def _the_one(self, what, need):
        names = [n for n, m in self.sides.items() if need(m) is not None]
        if len(names) > 1:
            raise ValueError(f"only one of two mixers side by side may need {what}")
        return names[0] if names else None

    @property
    def graph_safe(self) -> bool:
        return all(m.graph_safe for m in self.sides.values())

    @property
    def launches_only(self) -> bool:
        return all(m.launches_only for m in self.sides.values())

    def parameters(self):
        return {f"{n}.{k}": v for n, m in self.sides.items() for k, v in m.parameters().items()}

    def bind(self, tensors) -> None:
        super().bind(tensors)
        self.weights = {}
        outs, firsts = [], []
        for n, m in self.sides.items():
            m.bind({k: tensors[f"{n}.{k}"] for k in m.parameters()})
            outs.append(m.weights.pop("wo"))
            if self.in_weight:
                firsts.append(m.weights.pop(m.in_weight))
            self.weights.update({f"{n}.{k}": t for k, t in m.weights.items()})
            if m.has_out_bias:
                self.out_bias = m.out_bias
        self.weights["wo"] = torch.cat(outs, dim=1).contiguous()
        if self.in_weight:
            self.weights["win"], self.in_starts = stack_products(firsts)
            self.in_width = self.weights["win"].shape[0]

    def cache_need(self):
        return self.sides[self.cached].cache_need() if self.cached else None

    def state_need(self):
        return self.sides[self.stateful].state_need() if self.stateful else None

    def forward(self, ctx, x1, out, cache, state, z=None) -> None:
        left, right = self.sides["left"], self.sides["right"]
        wide = left.rows_width + right.rows_width
        rows = ctx.scratch("side.rows", (x1.shape[0], wide), self.dtype)
        if self.in_weight and z is None:
            z = ctx.scratch("side.z", (x1.shape[0], self.in_width), self.dtype)
            matmul_nt(x1, self.weights["win"], z)
        parts = (rows[:, :left.rows_width], rows[:, left.rows_width:])
        for i, ((n, m), part) in enumerate(zip(self.sides.items(), parts)):
            first = {} if z is None else {"z": z[:, self.in_starts[i]:self.in_starts[i] + m.in_width]}
            m.forward_rows(ctx, x1, part, cache if n == self.cached else None, state if n == self.stateful else None, **first)
        matmul_nt(rows, self.weights["wo"], out)
