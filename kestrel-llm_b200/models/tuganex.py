"""The Tuganex decoder assembled from parts.

The embedded tokens start the float32 stream.  Layers run in the order the configuration lists them; each is a
`PostNormBlock`: a sublayer reads the stream itself, its result is normed and then added.  A layer's mixer is one of

* ``attention``: `DifferentialAttention` over all earlier tokens - two softmax maps a head over the same values, the
  second subtracted from the first with a learned weight; q and k normed per head and map, rotate-half rotation of a
  head's first dimensions; with ``kv_from`` over the keys and values an earlier layer of the same step wrote;
* ``retention``: `RetentionMixer` - linear attention with a fixed decay per head, rotated q and k, a SiLU gate.

Feed-forward: none, `DenseMLP` with biases and the xIELU activation, or `SoftmaxRoutedExperts` (softmax router with a
correction per output and groups, SiLU-gated experts, identity experts, a gated expert that every token takes).  A final
RMSNorm and the output head.  Checkpoint tensors: ``embed``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*``,
``l<i>.mlp.*``, ``final.norm``, ``head``.
"""
from __future__ import annotations

import torch

from ..config.registry import register_architecture
from ..config.tuganex_config import NAME, DenseSpec, DifferentialSpec, MoeSpec, RetentionSpec, TuganexConfig
from ..parts import (DenseMLP, DifferentialAttention, LMHead, PostNormBlock, RetentionMixer, RMSNorm, RotaryHalf, SoftmaxRoutedExperts,
                     TokenEmbedding)
from .decoder import DecoderModel, LayerCall


def build_tuganex(config: TuganexConfig, dtype: torch.dtype, device) -> DecoderModel:
    c = config
    W, eps = c.hidden_size, c.norm_eps
    blocks, order, cache_of, optional = [], [], {}, []
    for i, layer in enumerate(c.layers):
        p, m = f"l{i}.", layer.mixer
        position = RotaryHalf(m.dim, m.rot.base, device, rotary_dim=m.rot.dims, exact=True) if m.rot is not None else None
        own = True
        if isinstance(m, DifferentialSpec):
            own = m.kv_from is None
            mixer = DifferentialAttention(W, m.heads, m.kv_heads, m.dim, m.vdim, dtype, device, p + "mix.", m.scale, eps, m.diff,
                                          position=position, own_kv=own)
        else:
            assert isinstance(m, RetentionSpec)
            mixer = RetentionMixer(W, m.heads, m.dim, m.vdim, m.decay, eps, dtype, device, p + "mix.", position=position)
        if own:
            cache_of[i] = len(cache_of)
        order.append(LayerCall(block=i, cache=cache_of[i if own else m.kv_from], writes_cache=own))
        f, norm2 = layer.mlp, None
        if f is None:
            ffn = None
            optional.append(p + "norm2")        # a layer without feed-forward has no use for it
        else:
            norm2 = RMSNorm(W, eps, device, p + "norm2")
            if isinstance(f, DenseSpec):
                ffn = DenseMLP(W, f.ff, dtype, device, p + "mlp.", activation="xielu", bias=True)
            else:
                assert isinstance(f, MoeSpec)
                ffn = SoftmaxRoutedExperts(W, f.ff, f.experts, f.top, dtype, device, p + "mlp.", identity=f.identity, groups=f.groups,
                                           keep=f.keep, shared_inner=f.shared_ff)
        blocks.append(PostNormBlock(mixer, RMSNorm(W, eps, device, p + "norm1"), ffn, norm2, dtype))
    return DecoderModel(c, dtype, device, TokenEmbedding(c.vocab_size, W, dtype, device, "embed"), None, blocks, order,
                        RMSNorm(W, eps, device, "final.norm"), LMHead(c.vocab_size, W, dtype, device, "head"), optional_tensors=optional)


register_architecture(NAME, TuganexConfig, build_tuganex)
