"""Gated feed-forward: y = W_down (silu(W_gate x) * W_up x), silu(z) = z / (1 + exp(-z))
(reference: st.c:8904-8914, st.c:3605-3607); with a ``limit`` L the bounded form W_down (g sigmoid(1.702 g) (u + 1)),
g = min(W_gate x, L), u = clamp(W_up x, -L, L).  Gate and up are one fused product.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from ..csrc import ops
from .base import FeedForward, WeightSlot
from .linear import Linear


class GatedMLP(FeedForward):
    graph_safe = True

    def __init__(self, width: int, intermediate: int, dtype: torch.dtype, device, prefix: str,
                 activation: str = "silu", names=("gate_proj.weight", "up_proj.weight", "down_proj.weight"), cut_few: bool = False,
                 limit: float = 0.0):
        if activation != "silu":
            raise ValueError(f"activation '{activation}' has no kernel; only 'silu'")
        self.width, self.intermediate = width, intermediate
        self.prefix, self.names = prefix, names
        self.dtype = dtype
        self.cut_few = cut_few               # a narrow one beside routed experts: few tokens take the product cut along K
        self.limit = float(limit)            # 0: none
        if self.limit < 0:
            raise ValueError("a bound on the gate and the up values is positive, or 0 for none")
        if cut_few or self.limit:
            self.emit = None                 # the step program has the uncut, unbounded form
        self.gate_up = Linear(width, 2 * intermediate, dtype, device)
        self.down = Linear(intermediate, width, dtype, device)

    def weight_slots(self) -> List[WeightSlot]:
        p, ff, (gate, up, down) = self.prefix, self.intermediate, self.names
        return [WeightSlot(p + gate, self.gate_up.weight[:ff]),
                WeightSlot(p + up, self.gate_up.weight[ff:]),
                WeightSlot(p + down, self.down.weight)]

    def forward(self, x: torch.Tensor, batch, residual: Optional[torch.Tensor] = None) -> Optional[ops.Partials]:
        act = ops.gate_up_swiglu(x, self.gate_up.weight, self.intermediate, weights_static=True, cut_few=self.cut_few,
                                 limit=self.limit)
        return self.down.forward(act, residual=residual)

    def emit(self, prog, x: int, residual: Optional[int]) -> int:
        act = prog.gate_up_swiglu(x, self.gate_up.weight, self.intermediate)
        return self.down.emit(prog, act, residual=residual, phase="down")


class DenseMLP(FeedForward):
    """Feed-forward without a gate: y = W_down act(W_up x), ``activation`` "relu2" (the square of
    relu), "silu", "tanh", "gelu" (the exact one, with erf), "gelu_tanh" or "xielu" (z^2 above zero, exp(z) - 1 - z
    below it, each times a learned number, plus z / 2; the checkpoint's two numbers are ``act_name``).  ``bias``: both projections
    have one."""
    graph_safe = True

    def __init__(self, width: int, intermediate: int, dtype: torch.dtype, device, prefix: str, activation: str = "relu2",
                 names=("up", "down"), bias: bool = False, act_name: str = "act"):
        if activation not in ("relu2", "silu", "tanh", "gelu", "gelu_tanh", "xielu"):
            raise ValueError(f"activation '{activation}' has no kernel; one of 'relu2', 'silu', 'tanh', 'gelu', 'gelu_tanh', 'xielu'")
        self.width, self.intermediate, self.activation = width, intermediate, activation
        self.prefix, self.names, self.dtype = prefix, names, dtype
        self.up = Linear(width, intermediate, dtype, device, bias=bias)
        self.down = Linear(intermediate, width, dtype, device, bias=bias)
        self.act_name = act_name
        self.act_params = torch.empty((2,), dtype=torch.float32, device=device) if activation == "xielu" else None

    def weight_slots(self) -> List[WeightSlot]:
        slots = []
        for name, proj in zip(self.names, (self.up, self.down)):
            slots.append(WeightSlot(self.prefix + name, proj.weight))
            if proj.bias is not None:
                slots.append(WeightSlot(self.prefix + name + ".b", proj.bias, "bias"))
        if self.act_params is not None:
            slots.append(WeightSlot(self.prefix + self.act_name, self.act_params, "bias"))
        return slots

    def forward(self, x: torch.Tensor, batch) -> ops.Partials:
        # many tokens in bfloat16: the activation is the up product's epilogue; otherwise its slices are summed and activated
        return self.down.forward(ops.linear_act(x, self.up.weight, self.activation, weights_static=True, bias=self.up.bias,
                                               act_params=self.act_params))
