"""Retention: linear attention with a fixed decay per head, without softmax or denominator, carried from token to token as a
matrix per head in the request's state slot (float32, zero at admission).

    q = W_q h,  k = W_k h  [H, d],  v = W_v h  [H, dv],  gate logits W_g h  [H dv]         one fused product, no biases
    q, k turned by position (rotate-half pairs of a head's first dimensions), then k times d^-1/2
    S_t = decay_h S_{t-1} + k_t v_t^T,   o_t = S_t^T q_t                                   per head
    o <- o / sqrt(mean(o^2) + eps) per head (no weight),   y = W_o (o * silu(gate logits))

``decay`` lists a number per head.  Steps of at most `STEP_TOKENS` tokens per request run one kernel between the two products; in
bfloat16 steps that bring a request `CHUNKED_FROM` tokens or more run in chunks on the tensor cores; the rest runs on the sequential
scan that the other recurrences share.
"""
from __future__ import annotations

from typing import List, Optional, Sequence

import torch

from ..csrc import ops
from .base import FixedStateSpec, Mixer, PositionEncoding, WeightSlot
from .linear import Linear


class RetentionMixer(Mixer):
    STEP_TOKENS = 4
    CHUNKED_FROM = 32
    chunked = True             # tests switch the chunked form and the one-kernel form off to hold the forms against each other
    one_kernel = True
    graph_safe = True          # forward launches kernels over device tensors of the batch only

    def __init__(self, width: int, heads: int, dim: int, v_dim: int, decay: Sequence[float], norm_eps: float, dtype: torch.dtype, device,
                 prefix: str, position: Optional[PositionEncoding] = None, names=("q", "k", "v", "g", "o")):
        if dim > 256:
            raise ValueError(f"key size {dim}: the scan holds up to 256 key channels a column")
        if len(decay) != heads:
            raise ValueError(f"{len(decay)} decays for {heads} heads")
        self.width, self.H, self.d, self.dv = width, heads, dim, v_dim
        self.eps, self.dtype, self.prefix, self.names = float(norm_eps), dtype, prefix, names
        self.qk, self.vg = heads * dim, heads * v_dim
        self.col_g = 2 * self.qk + self.vg
        self.in_proj = Linear(width, 2 * self.qk + 2 * self.vg, dtype, device)         # columns [q | k | v | gate]
        self.out = Linear(self.vg, width, dtype, device)
        self.rotation = position.rotary() if position is not None else None
        # decay^n for the distances inside a chunk, made once in float64
        powers = torch.tensor([[float(x) ** n for n in range(65)] for x in decay], dtype=torch.float64).to(torch.float32)
        self.powers = powers.to(device) if torch.device(device).type != "meta" else torch.empty_like(powers, device=device)
        self.decay = torch.tensor([float(x) for x in decay], dtype=torch.float32)
        self.decay = self.decay.to(device) if torch.device(device).type != "meta" else torch.empty_like(self.decay, device=device)

    def cache_spec(self) -> FixedStateSpec:
        return FixedStateSpec((self.H * self.d * self.dv,), torch.float32)

    def weight_slots(self) -> List[WeightSlot]:
        p, w, (q, k, v, g, o) = self.prefix, self.in_proj.weight, self.names
        return [WeightSlot(p + q, w[:self.qk]), WeightSlot(p + k, w[self.qk:2 * self.qk]), WeightSlot(p + v, w[2 * self.qk:self.col_g]),
                WeightSlot(p + g, w[self.col_g:]), WeightSlot(p + o, self.out.weight)]

    def forward(self, x: torch.Tensor, batch, cache) -> ops.Partials:
        H, d, dv = self.H, self.d, self.dv
        fused = self.in_proj.forward(x)
        y = torch.empty((x.shape[0], self.vg), dtype=self.dtype, device=x.device)
        if batch.max_count <= self.STEP_TOKENS and dv <= 256 and self.one_kernel:
            ops.retention_step(fused, batch.positions, self.rotation, self.decay, cache.state, batch, self.eps, y, H, d, dv)
        elif self.dtype == torch.bfloat16 and not batch.captured and batch.max_count >= self.CHUNKED_FROM and self.chunked and \
                d % 8 == 0 and dv % 8 == 0 and dv <= 256:
            q, k, v, _ = ops.retention_prepare(fused, batch.positions, self.rotation, self.decay, torch.bfloat16, H, d, dv, with_decay=False)
            ops.retention_chunks(q, k, v, self.powers, fused, self.col_g, cache.state, batch, self.eps, y, H, d, dv)
        else:
            q, k, v, w = ops.retention_prepare(fused, batch.positions, self.rotation, self.decay, torch.float32, H, d, dv)
            o = ops.recurrence_scan(q, w, k, v, None, None, cache.state, 0, batch, H, d, dv)
            ops.head_norm_gate(o, None, self.eps, fused, self.col_g, y, H, dv, gate_act="silu")
        return self.out.forward(y)
