"""The Fasanex decoder assembled from parts.

The embedded tokens times a constant start the float32 stream.  Layers run in the order the configuration lists them; each is a
`SandwichBlock` without gates: a norm in front of a sublayer and another on its result, which is then added; all norms of the model
width store their weight as its distance from one.  A layer's mixer is one of

* ``mamba2``: `StateSpaceMixer` - a recurrence with a scalar decay per head behind a short convolution, gated, normed in parts;
* ``parallel``: `JoinedMixers` of a `GatedWindowAttention` - a window, rotated heads behind a short convolution, keys that are their
  own values, capped scores, a gate per element - and a `TimeMixRecurrence`, their results weighted and added;
* ``delta``: `HeadDeltaMixer` - the gated delta rule with one decay per head.

Feed-forward: none, or `GatedMLP` with the bounded activation.  A final norm and the output head.  Checkpoint tensors: ``embed``,
``l<i>.norm1``, ``norm1b``, ``norm2``, ``norm2b``, ``l<i>.mix.*``, ``l<i>.mlp.{gate,up,down}``, ``final.norm``, ``head``.
"""
from __future__ import annotations

import torch

from ..config.fasanex_config import NAME, FasanexConfig, HeadDeltaSpec, JoinedSpec, StateSpaceSpec
from ..config.registry import register_architecture
from ..parts import (GatedMLP, GatedWindowAttention, HeadDeltaMixer, JoinedMixers, LMHead, RampScaling, RMSNorm, RotaryHalf, SandwichBlock,
                     StateSpaceMixer, TimeMixRecurrence, TokenEmbedding)
from .decoder import DecoderModel, LayerCall


def _attention(a, width: int, eps: float, dtype: torch.dtype, device, prefix: str) -> GatedWindowAttention:
    position = None
    if a.rot is not None:
        s = a.rot.scaling
        ramp = RampScaling(s.factor, s.original, s.fast, s.slow, a.rot.dims, a.rot.base) if s is not None else None
        position = RotaryHalf(a.dim, a.rot.base, device, rotary_dim=a.rot.dims, scale=ramp.magnitude if ramp is not None else 1.0, scaling=ramp,
                              exact=True)
    return GatedWindowAttention(width, a.heads, a.kv_heads, a.dim, a.dim, dtype, device, prefix, a.scale, eps, window=a.window, head_gate=False,
                                element_gate=True, softcap=a.softcap, qk_norm="head", head_norm_weight=True, position=position, conv_taps=a.conv,
                                values_from_keys=True, out_proj=False)


def build_fasanex(config: FasanexConfig, dtype: torch.dtype, device) -> DecoderModel:
    c = config
    W, eps = c.hidden_size, c.norm_eps
    blocks, optional = [], []

    def norm(name: str) -> RMSNorm:
        return RMSNorm(W, eps, device, name, around_zero=True)
    for i, layer in enumerate(c.layers):
        p, m = f"l{i}.", layer.mixer
        if isinstance(m, StateSpaceSpec):
            mixer = StateSpaceMixer(W, m.heads, m.vdim, m.state, m.groups, m.norm_groups, m.conv, eps, dtype, device, p + "mix.")
        elif isinstance(m, JoinedSpec):
            if not m.right.decay_rank:
                raise ValueError(f"layer {i}: the rank of the decay's projection is unknown (FasanexConfig.with_tensor_shapes)")
            left = _attention(m.left, W, eps, dtype, device, p + "mix.left.")
            right = TimeMixRecurrence(W, m.right.heads, m.right.dim, m.right.decay_rank, eps, dtype, device, p + "mix.right.", out_proj=False)
            mixer = JoinedMixers(left, right, W, m.left_scale, m.right_scale, dtype, device, p + "mix.")
        else:
            assert isinstance(m, HeadDeltaSpec)
            mixer = HeadDeltaMixer(W, m.heads, m.kv_heads, m.dim, m.vdim, m.conv, eps, dtype, device, p + "mix.")
        ffn = norm2 = norm2b = None
        if layer.mlp is not None:
            ffn = GatedMLP(W, layer.mlp.ff, dtype, device, p + "mlp.", names=("gate", "up", "down"), limit=layer.mlp.limit)
            norm2, norm2b = norm(p + "norm2"), norm(p + "norm2b")
        else:
            optional += [p + "norm2", p + "norm2b"]         # a layer without feed-forward has no use for them
        blocks.append(SandwichBlock(norm(p + "norm1"), mixer, norm(p + "norm1b"), None, norm2, ffn, norm2b, None, dtype, p))
    for block, after in zip(blocks, blocks[1:]):
        block.following = after.norm1                       # the last add of a layer makes the norm of the next one
    order = [LayerCall(block=i, cache=i) for i in range(len(blocks))]
    return DecoderModel(c, dtype, device, TokenEmbedding(c.vocab_size, W, dtype, device, "embed", scale=c.embedding_scale), None, blocks, order,
                        norm("final.norm"), LMHead(c.vocab_size, W, dtype, device, "head"), optional_tensors=optional)


register_architecture(NAME, FasanexConfig, build_fasanex)
