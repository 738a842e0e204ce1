"""State-space mixer with a scalar decay per head (Mamba-2).

With h the mixer's input, H heads of P value channels, G groups of N state channels, inner = H P:

    z | x | B | C | dt = W_in h                                            widths inner, inner, G N, G N, H
    x, B, C <- silu(conv(.) + b)                                           a causal convolution over time per channel
    dt <- softplus(dt + dt_bias)
    S_t = exp(-exp(A_log) dt) S_{t-1} + dt B_t x_t^T,   y_t = S_t^T C_t + D x_t     per head with its group's B and C, S [N, P] from zero
    out = W_o ( norm(y * silu(z)) * w )                                    the norm over `norm_groups` equal parts of the inner channels

The state S and the convolution's last taps - 1 inputs live in the request's state slot, float32; step sizes, decays, recurrence,
gate and norm are float32.  Steps of at most `STEP_TOKENS` tokens per request run one kernel between the input product and the norm; in
bfloat16 longer ones run in chunks on the tensor cores; the rest runs on the sequential scan that the other recurrences share.
"""
from __future__ import annotations

from typing import List

import torch

from ..csrc import ops
from .base import FixedStateSpec, Mixer, WeightSlot
from .linear import Linear


class StateSpaceMixer(Mixer):
    STEP_TOKENS = 4
    chunked = True             # tests switch the chunked form and the one-kernel form off to hold the forms against each other
    one_kernel = True
    graph_safe = True          # forward launches kernels over device tensors of the batch only

    def __init__(self, width: int, heads: int, value_dim: int, state: int, groups: int, norm_groups: int, taps: int, norm_eps: float,
                 dtype: torch.dtype, device, prefix: str):
        if heads % groups:
            raise ValueError(f"{heads} heads are not a multiple of {groups} groups")
        if (heads * value_dim) % norm_groups:
            raise ValueError(f"{heads * value_dim} channels do not divide into {norm_groups} parts")
        if state > 256:
            raise ValueError(f"{state} state channels: the scan holds up to 256")
        if not 1 <= taps <= 9:
            raise ValueError(f"{taps} taps: the convolution takes 1 to 9")
        self.width, self.H, self.P, self.N, self.G, self.parts, self.taps = width, heads, value_dim, state, groups, norm_groups, taps
        self.eps, self.dtype, self.prefix = float(norm_eps), dtype, prefix
        self.inner = heads * value_dim
        self.C = self.inner + 2 * groups * state               # channels that pass the convolution: x | B | C
        self.col_dt = self.inner + self.C
        self.in_proj = Linear(width, self.inner + self.C + heads, dtype, device)
        self.out = Linear(self.inner, width, dtype, device)
        f32 = dict(dtype=torch.float32, device=device)
        self.conv_w, self.conv_b = torch.empty((taps, self.C), **f32), torch.empty((self.C,), **f32)
        self.dt_bias, self.A_log, self.D = (torch.empty((heads,), **f32) for _ in range(3))
        self.norm_w = torch.empty((self.inner,), **f32)
        self.tail_off = (heads * state * value_dim + 3) // 4 * 4       # the slot: S [H, N, P], then the convolution's tail [taps - 1, C]
        self.state_size = (self.tail_off + (taps - 1) * self.C + 3) // 4 * 4

    def cache_spec(self) -> FixedStateSpec:
        return FixedStateSpec((self.state_size,), torch.float32)

    def weight_slots(self) -> List[WeightSlot]:
        p = self.prefix
        return [WeightSlot(p + "in", self.in_proj.weight), WeightSlot(p + "conv", self.conv_w.t(), "bias"), WeightSlot(p + "conv.b", self.conv_b, "bias"),
                WeightSlot(p + "dt_bias", self.dt_bias, "bias"), WeightSlot(p + "A_log", self.A_log, "bias"), WeightSlot(p + "D", self.D, "norm"),
                WeightSlot(p + "norm", self.norm_w, "norm"), WeightSlot(p + "o", self.out.weight)]

    def forward(self, x: torch.Tensor, batch, cache) -> ops.Partials:
        H, G, N, P = self.H, self.G, self.N, self.P
        T, dev = x.shape[0], x.device
        fused = self.in_proj.forward(x)
        y = torch.empty((T, self.inner), dtype=self.dtype, device=dev)
        if batch.max_count <= self.STEP_TOKENS and P <= 256 and self.one_kernel:
            o = ops.ssm_step(fused, 0, self.inner, self.col_dt, self.conv_w, self.conv_b, self.dt_bias, self.A_log, self.D, cache.state, self.tail_off,
                             batch, H, G, N, P)
            ops.part_norm(o, self.norm_w, self.eps, y, self.parts)
            return self.out.forward(y)
        chunks = self.dtype == torch.bfloat16 and not batch.captured and self.chunked and N % 8 == 0 and P % 8 == 0 and P <= 256 and fused.width % 2 == 0
        act = torch.empty((T, self.C), dtype=torch.bfloat16 if chunks else torch.float32, device=dev)
        ops.short_conv(fused, self.conv_w, self.conv_b, cache.state, self.tail_off, batch, act, col0=self.inner)
        if chunks:
            o = ops.ssm_chunks(act, fused, 0, self.col_dt, self.dt_bias, self.A_log, self.D, cache.state, batch, H, G, N, P)
            ops.part_norm(o, self.norm_w, self.eps, y, self.parts)
        else:
            r, w, k, v = ops.ssm_expand(act, fused, self.col_dt, self.dt_bias, self.A_log, H, G, N, P)
            o = ops.recurrence_scan(r, w, k, v, None, None, cache.state, 0, batch, H, N, P)
            ops.ssm_out(o, act, self.D, fused, 0, self.norm_w, self.eps, y, H, G, N, P, self.parts)
        return self.out.forward(y)
