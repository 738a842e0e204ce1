"""Two mixers side by side on the same input: each one's output is RMS-normed over the model
width with a weight of its own, and the mixer's result is their weighted sum,

    y = mix * (rmsnorm(left(h)) * w_left + rmsnorm(right(h)) * w_right)          (mix = 1/2: the mean)

The two keep what they keep - pages of keys and values, a state slot - in ONE cache layer: its
spec is a `CombinedSpec` of theirs, and both are handed the layer's `LayerCache`, of which each
uses its own part.

`JoinedMixers` is the arrangement without norms: y = left_scale * left(h) + right_scale * right(h).  Both mixers end in a projection of
their concatenated heads, so the two projections are ONE product over the heads of both, [left_scale a | right_scale b] times
[W_left | W_right]: each mixer leaves its heads, times its factor (a float32 step of its last kernel), in its columns of one matrix.
"""
from __future__ import annotations

from typing import List

import torch

from ..csrc import ops
from .base import CacheSpec, CombinedSpec, FixedStateSpec, Mixer, PagedKVSpec, WeightSlot, paged_part, state_part
from .linear import Linear


class ParallelMixers(Mixer):
    def __init__(self, left: Mixer, right: Mixer, width: int, norm_eps: float, device, prefix: str, names=("left.out", "right.out"),
                 mix: float = 0.5):
        self.left, self.right, self.width = left, right, width
        self.eps, self.mix, self.prefix, self.names = float(norm_eps), float(mix), prefix, names
        self.w_left = torch.empty((width,), dtype=torch.float32, device=device)
        self.w_right = torch.empty((width,), dtype=torch.float32, device=device)
        specs = [sp for sp in (left.cache_spec(), right.cache_spec()) if sp is not None]
        paged = [sp for sp in specs if isinstance(sp, PagedKVSpec)]
        state = [sp for sp in specs if isinstance(sp, FixedStateSpec)]
        if len(paged) > 1 or len(state) > 1 or len(paged) + len(state) != len(specs):
            raise ValueError("two mixers side by side share one cache layer: at most one of them keeps pages and at most one a state")
        self._spec: CacheSpec = specs[0] if len(specs) == 1 else (CombinedSpec(paged[0], state[0]) if specs else None)

    @property
    def graph_safe(self) -> bool:
        return bool(getattr(self.left, "graph_safe", False) and getattr(self.right, "graph_safe", False))

    def cache_spec(self) -> CacheSpec:
        return self._spec

    def weight_slots(self) -> List[WeightSlot]:
        return self.left.weight_slots() + self.right.weight_slots() + [WeightSlot(self.prefix + self.names[0], self.w_left, "norm"),
                                                                      WeightSlot(self.prefix + self.names[1], self.w_right, "norm")]

    def forward(self, x: torch.Tensor, batch, cache) -> ops.Partials:
        a = self.left.forward(x, batch, cache)
        b = self.right.forward(x, batch, cache)
        for p in (a, b):
            if p.bias is not None:
                raise ValueError("a mixer that runs beside another hands over its product without a pending bias")
        return ops.combine_normed(a, self.w_left, b, self.w_right, self.eps, self.mix)


class JoinedMixers(Mixer):
    """``left`` and ``right`` offer `heads_into(x, batch, cache, out, scale)`` and ``out_features``, have no output projection of their own,
    and keep their state from ``state_off`` of the request's slot on (set here: the left one's first, then the right one's)."""

    def __init__(self, left: Mixer, right: Mixer, width: int, left_scale: float, right_scale: float, dtype: torch.dtype, device, prefix: str,
                 names=("left.o", "right.o")):
        self.left, self.right = left, right
        self.left_scale, self.right_scale = float(left_scale), float(right_scale)
        self.dtype, self.prefix, self.names = dtype, prefix, names
        self.out = Linear(left.out_features + right.out_features, width, dtype, device)
        paged = [sp for sp in (paged_part(m.cache_spec()) for m in (left, right)) if sp is not None]
        if len(paged) > 1:
            raise ValueError("two mixers side by side share one cache layer: at most one of them keeps pages")
        size = 0
        for m in (left, right):
            sp = state_part(m.cache_spec())
            if sp is None:
                continue
            if len(sp.shape) != 1 or sp.dtype != torch.float32:
                raise ValueError("mixers side by side keep their state as a vector of float32 each")
            m.state_off = size
            size += (sp.shape[0] + 3) // 4 * 4             # every part starts on a 16-byte boundary
        state = FixedStateSpec((size,), torch.float32) if size else None
        self._spec: CacheSpec = CombinedSpec(paged[0], state) if paged and state else (paged[0] if paged else state)

    @property
    def graph_safe(self) -> bool:
        return bool(getattr(self.left, "graph_safe", False) and getattr(self.right, "graph_safe", False))

    def cache_spec(self) -> CacheSpec:
        return self._spec

    def weight_slots(self) -> List[WeightSlot]:
        n = self.left.out_features
        return self.left.weight_slots() + self.right.weight_slots() + [WeightSlot(self.prefix + self.names[0], self.out.weight[:, :n]),
                                                                      WeightSlot(self.prefix + self.names[1], self.out.weight[:, n:])]

    def forward(self, x: torch.Tensor, batch, cache) -> ops.Partials:
        n = self.left.out_features
        heads = torch.empty((x.shape[0], self.out.in_features), dtype=self.dtype, device=x.device)
        self.left.heads_into(x, batch, cache, heads[:, :n], self.left_scale)
        self.right.heads_into(x, batch, cache, heads[:, n:], self.right_scale)
        return self.out.forward(heads)
