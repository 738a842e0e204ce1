"""Time mixing (the RWKV form of linear attention): every projection reads its own blend of a token and the one before it, and the
state decays per head and key channel at a rate that depends on the token.

With h the mixer's input, h' the previous token's (zeros for a request's first), s one of r, k, v, g, w, H heads of size d:

    x_s = h + (h' - h) * mu_s;     r, k, v = W_r x_r, W_k x_k, W_v x_v;     gate = silu(W_g x_g)
    w = exp(-exp(W_w2 tanh(W_w1 x_w) + w0))                                        per head and key channel
    o_t = (S_{t-1} + diag(u) k_t v_t^T)^T r_t;     S_t = diag(w_t) S_{t-1} + k_t v_t^T     per head, S [d, d] from zero
    y = W_o ( o / sqrt(mean(o^2) + eps) per head * w_norm * gate )

The state S and the last h live in the request's state slot, float32; what enters the recurrence is float32.  The five products of the blends
are one launch where the product allows it (`ops.linear_groups`).  Steps of at most `STEP_TOKENS` tokens
per request run one kernel between the products; in bfloat16 longer ones run in chunks on the tensor cores; the rest runs on the sequential
scan that the other recurrences share.
"""
from __future__ import annotations

from typing import List

import torch

from ..csrc import ops
from .base import FixedStateSpec, Mixer, WeightSlot
from .linear import Linear


class TimeMixRecurrence(Mixer):
    STEP_TOKENS = 4
    chunked = True             # tests switch the chunked form and the one-kernel form off to hold the forms against each other
    one_kernel = True
    graph_safe = True          # forward launches kernels over device tensors of the batch only

    def __init__(self, width: int, heads: int, dim: int, decay_rank: int, norm_eps: float, dtype: torch.dtype, device, prefix: str,
                 out_proj: bool = True):
        if dim > 256:
            raise ValueError(f"key size {dim}: the scan holds up to 256 key channels a column")
        if decay_rank <= 0:
            raise ValueError("the rank of the decay's two-step projection must be positive")
        self.width, self.H, self.d, self.rank = width, heads, dim, decay_rank
        self.eps, self.dtype, self.prefix = float(norm_eps), dtype, prefix
        n = self.out_features = heads * dim
        # rows r | k | v | g | the decay's first step, each over its own blend; a rank beyond the others' size stays a product of its own
        self.w1 = Linear(width, decay_rank, dtype, device) if decay_rank > n else None
        self.proj = Linear(width, 4 * n + (decay_rank if self.w1 is None else 0), dtype, device)
        self.w2 = Linear(decay_rank, n, dtype, device)
        self.out = Linear(n, width, dtype, device) if out_proj else None
        f32 = dict(dtype=torch.float32, device=device)
        self.mu = torch.empty((5, width), **f32)                 # r, k, v, g, w
        self.w0 = torch.empty((n,), **f32)
        self.u = torch.empty((heads, dim), **f32)
        self.norm_w = torch.empty((n,), **f32)
        self.state_off = 0         # where the mixer's state starts in the request's slot: S [H, d, d], then the last h
        self.last_off = (heads * dim * dim + 3) // 4 * 4
        self.state_size = self.last_off + width

    def cache_spec(self) -> FixedStateSpec:
        return FixedStateSpec((self.state_size,), torch.float32)

    def weight_slots(self) -> List[WeightSlot]:
        p, w, n = self.prefix, self.proj.weight, self.out_features
        slots = [WeightSlot(p + "mu." + s, self.mu[i], "unit") for i, s in enumerate("rkvgw")]
        slots += [WeightSlot(p + s, w[i * n:(i + 1) * n]) for i, s in enumerate("rkvg")]
        slots += [WeightSlot(p + "w1", w[4 * n:] if self.w1 is None else self.w1.weight), WeightSlot(p + "w2", self.w2.weight), WeightSlot(p + "w0", self.w0, "bias"),
                  WeightSlot(p + "u", self.u, "bias"), WeightSlot(p + "norm", self.norm_w, "norm")]
        if self.out is not None:
            slots.append(WeightSlot(p + "o", self.out.weight))
        return slots

    def forward(self, x: torch.Tensor, batch, cache) -> ops.Partials:
        y = torch.empty((x.shape[0], self.out_features), dtype=self.dtype, device=x.device)
        self.heads_into(x, batch, cache, y, 1.0)
        return self.out.forward(y)

    def heads_into(self, x: torch.Tensor, batch, cache, out: torch.Tensor, scale: float) -> None:
        """Everything in front of the output projection, times ``scale``, into ``out`` [T, H d]."""
        H, d, n = self.H, self.d, self.out_features
        blends = ops.token_shift(x, self.mu, cache.state, self.state_off + self.last_off, batch)
        if self.w1 is None:
            p = ops.linear_groups(blends, self.proj.weight, n)
            first = ops.partial_columns_act(p, 4 * n, self.rank, self.dtype, "tanh")
        else:
            p = ops.linear_groups(blends[:4], self.proj.weight, n)
            first = ops.linear_act(blends[4], self.w1.weight, "tanh", weights_static=True)
        z = self.w2.forward(first)
        last = self.state_off + self.last_off
        rest = (p, z, self.w0, self.u, self.norm_w, self.eps, scale, x, cache.state, self.state_off, last, batch, out, H, d)
        if batch.max_count <= self.STEP_TOKENS and self.one_kernel:
            ops.time_mix_step(*rest)
        elif self.dtype == torch.bfloat16 and not batch.captured and self.chunked and d % 8 == 0 and d <= 128 and p.width % 4 == 0 and \
                out.stride(0) % 2 == 0 and out.data_ptr() % 4 == 0:
            ops.time_mix_chunks(*rest)
        else:
            r, w, k, v = ops.time_mix_gates(p, z, self.w0, n, x, cache.state, last, batch)
            o = ops.recurrence_scan_bonus(r, w, k, v, self.u, cache.state, self.state_off, batch, H, d, d)
            ops.head_norm_gate(o, self.norm_w, self.eps, p, 3 * n, out, H, d, gate_act="silu", scale=scale)
