"""Grouped-query differential attention over the paged cache: every head has two softmax maps, with queries and keys of their
own, over the same values, and the second is subtracted from the first.

    q = W_q h  [H, 2, d],  k = W_k h  [G, 2, d],  v = W_v h  [G, dv]        one fused product, no biases
    q, k <- RMS norm per head and map over d, weights [d] shared by all heads and maps, then turned by position
    a_i = softmax_j(q_i . k_ij * scale) v        map i = 1, 2; query head n uses key/value head n // (H / G)
    lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff                 one number a layer, from four learned vectors [d]
    o = a_1 - lambda a_2;   o <- o / sqrt(mean(o^2) + eps) * (1 - diff)     per head
    y = W_o o

A token's cache row holds both maps' keys, [k_1 | k_2], as ONE key of 2 d numbers, so a layer's pages are those of any grouped
attention with head sizes (2 d, dv).  A query of map i is that long too, zero in the other map's half: its dot product with a row is
its own map's score, and 2 H query heads over G key/value heads run on the attention kernels as they are - keys and values are read
once for both maps.  Their float32 outputs are combined by `ops.differential_combine`.  Steps with prompt portions of maps of 64
over values of 128 take the tcgen05 kernel (`ops.attention_tc_maps`), which works on the two maps as two row tiles, multiplies each
with its own half of the keys, and combines and norms the heads itself; a long key range is cut into slices there so that the few
tiles of a portion far into a context fill the chip.  Steps of few tokens share the keys out over CTAs; the kernel that merges the
shares combines and norms the heads.

A mixer built with ``own_kv=False`` has no key and value projections and attends over the pages that an earlier layer of the same
step wrote, with its own queries, lambda and scale.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from ..csrc import ops
from .base import Mixer, PagedKVSpec, PositionEncoding, WeightSlot
from .linear import Linear


class DifferentialAttention(Mixer):
    force_plain = False        # tests: bfloat16 through the plain kernel too, the twin of the tensor-core one
    tcgen05 = True             # tests: off, portions of maps of 64 over values of 128 stay on the mma.sync kernel
    decode = True              # tests: off, single tokens of 2 x 32 / 64 and 2 x 64 / 128 stay on the kernel of every other size
    TC_MIN_ROWS = 64           # a step whose longest portion has more rows (tokens x heads of a group) takes the tcgen05 kernel
    TC_SLICE = 512             # fewest keys a slice where a portion's key range is cut
    TC_SLICE_FILL = 148        # CTAs that the cut should reach: one an SM
    graph_safe = True          # forward launches kernels over device tensors of the batch only

    def __init__(self, width: int, heads: int, kv_heads: int, dim: int, v_dim: int, dtype: torch.dtype, device, prefix: str, scale: float,
                 norm_eps: float, diff: float, position: Optional[PositionEncoding] = None, own_kv: bool = True,
                 names=("q", "k", "v", "o"), norm_suffix: str = ".norm", lambda_names=("lq1", "lk1", "lq2", "lk2")):
        if heads % kv_heads:
            raise ValueError(f"{heads} query heads are not a multiple of {kv_heads} kv heads")
        if dim > 256 or v_dim > 256:
            raise ValueError(f"sizes {dim} / {v_dim} of a map and a value: the kernels take up to 256")
        self.width, self.heads, self.kv_heads, self.dim, self.v_dim = width, heads, kv_heads, dim, v_dim
        self.scale, self.norm_eps, self.diff, self.own_kv = float(scale), float(norm_eps), float(diff), own_kv
        self.prefix, self.names, self.norm_suffix, self.lambda_names, self.dtype = prefix, names, norm_suffix, lambda_names, dtype
        self.q_cols = heads * 2 * dim
        self.k_cols, self.v_cols = (kv_heads * 2 * dim, kv_heads * v_dim) if own_kv else (0, 0)
        self.proj = Linear(width, self.q_cols + self.k_cols + self.v_cols, dtype, device)
        self.out = Linear(heads * v_dim, width, dtype, device)
        self.rotation = position.rotary() if position is not None else None
        if self.rotation is not None and self.rotation.dim > dim:
            raise ValueError(f"{self.rotation.dim} rotated dimensions exceed the map's size {dim}")
        f32 = dict(dtype=torch.float32, device=device)
        self.q_norm = torch.empty((dim,), **f32)
        self.k_norm = torch.empty((dim,), **f32) if own_kv else None
        self.lambdas = [torch.empty((dim,), **f32) for _ in range(4)]           # lq1, lk1, lq2, lk2

    def cache_spec(self) -> PagedKVSpec:
        return PagedKVSpec(self.kv_heads, 2 * self.dim, v_head_dim=self.v_dim)

    def weight_slots(self) -> List[WeightSlot]:
        p, (nq, nk, nv, no), w = self.prefix, self.names, self.proj.weight
        k_end = self.q_cols + self.k_cols
        slots = [WeightSlot(p + nq, w[:self.q_cols])]
        if self.own_kv:
            slots += [WeightSlot(p + nk, w[self.q_cols:k_end]), WeightSlot(p + nv, w[k_end:]),
                      WeightSlot(p + nk + self.norm_suffix, self.k_norm, "norm")]
        slots += [WeightSlot(p + nq + self.norm_suffix, self.q_norm, "norm"), WeightSlot(p + no, self.out.weight)]
        return slots + [WeightSlot(p + n, t, "bias") for n, t in zip(self.lambda_names, self.lambdas)]

    def forward(self, x: torch.Tensor, batch, cache) -> ops.Partials:
        if cache.writable != self.own_kv:
            raise ValueError("a mixer with key and value projections writes its cache layer; one without reads another's")
        T, H, G, d, dv = x.shape[0], self.heads, self.kv_heads, self.dim, self.v_dim
        fused = self.proj.forward(x)
        table = batch.block_table(cache.group)
        o = torch.empty((T, H * dv), dtype=self.dtype, device=x.device)
        fast = self.dtype == torch.bfloat16 and not self.force_plain
        tc = fast and self.tcgen05 and (d, dv) == (64, 128) and not batch.captured and batch.max_count * (H // G) > self.TC_MIN_ROWS and \
            ops.attention_tc_supported(128, cache.page_size)
        q = torch.empty((T, 2 * H * d * (1 if tc else 2)), dtype=self.dtype, device=x.device)
        ops.attn_prepare_ex(fused, self.q_norm, self.k_norm, "head", self.norm_eps, batch.positions, batch.seq_of_token, table, cache.page_size,
                            cache.k, cache.v, q, None, H, G, d, dv, self.own_kv, rotation=self.rotation, maps=2, q_pad=not tc)
        if tc:
            # few tiles far into a long context: as many slices of the keys as fill the chip
            tiles = sum(-(-n * (H // G) // 128) for n in batch.counts)
            fill, slices, slice_len = self.TC_SLICE_FILL // max(1, tiles * G), 1, 1 << 30
            if fill >= 2 and batch.max_kv_len > 2 * self.TC_SLICE:
                per = -(-batch.max_kv_len // min(32, fill))
                slice_len = max(self.TC_SLICE, (per + 127) // 128 * 128)
                slices = -(-batch.max_kv_len // slice_len)
            ops.attention_tc_maps(q, cache.k, cache.v, o, batch, table, cache.page_size, H, G, d, dv, self.scale, self.lambdas, self.diff,
                                  self.norm_eps, slices, slice_len)
            return self.out.forward(o)
        if fast and self.decode and ops.attention_decode_maps(q, cache.k, cache.v, batch, table, cache.page_size, o, H, G, d, dv, self.scale,
                                                              self.lambdas, self.diff, self.norm_eps):
            return self.out.forward(o)
        window = fast and ops.attention_window_supported(2 * d, dv, 2 * H, G)
        if window and ops.attention_window_maps(q, cache.k, cache.v, batch, table, cache.page_size, o, H, G, d, dv, self.scale, self.lambdas,
                                                self.diff, self.norm_eps):
            return self.out.forward(o)
        a = torch.empty((T, 2 * H * dv), dtype=torch.float32, device=x.device)
        if window:
            ops.attention_window(q, cache.k, cache.v, batch, table, cache.page_size, a, 2 * H, G, 2 * d, dv, 0, 0, None, self.scale)
        else:           # float32, sizes that are no multiple of 8, and maps of more than 128
            ops.attention_plain_ex(q, cache.k, cache.v, batch.positions, batch.seq_of_token, table, cache.page_size, a, 2 * H, G, 2 * d, dv, 0, 0,
                                   None, self.scale)
        ops.differential_combine(a, *self.lambdas, self.diff, self.norm_eps, o, H, dv)
        return self.out.forward(o)
