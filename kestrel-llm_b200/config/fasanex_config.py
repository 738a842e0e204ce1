"""Typed configuration of the Fasanex decoder, read from its own ``config.json`` keys.

Top level: ``architecture`` (a string), ``vocab``, ``width``, ``norm.eps``, ``embedding.scale`` (absent: 1) and ``layers``, a list with one
entry per layer: ``type`` (which mixer), ``mixer`` (its sizes and constants) and ``mlp`` (``{"kind": "dense", "ff": n, "limit": x}``, or null).

* ``mamba2``: ``heads``, ``vdim``, ``state``, ``groups``, ``norm_groups``, ``conv`` (taps).
* ``parallel``: ``left`` - attention whose values are its keys: ``heads``, ``kv_heads``, ``dim`` (= ``vdim``), ``conv``, ``scale``,
  ``softcap`` (absent or null: none), ``mask.size`` (absent: every earlier token), ``rot`` (``dims``, ``base``, and optionally ``scaling``
  with ``factor``, ``original``, ``fast``, ``slow``; absent: no rotation) -, ``right`` - time mixing: ``heads``, ``dim``; the rank of its
  decay's two-step projection is the size of a checkpoint tensor (``decay_rank`` may name it; `with_tensor_shapes` fills it in) -,
  ``left_scale``, ``right_scale``.
* ``delta``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv``.

Every size and constant comes from the file; nothing is assumed equal between layers.
"""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Any, Dict, Optional, Tuple

from .korirax_config import RotSpec, _rot
from .model_config import ConfigError, ModelConfig
from .zidivik_config import _number, _pos_int

NAME = "Fasanex"

MAMBA2, PARALLEL, DELTA = "mamba2", "parallel", "delta"


@dataclass(frozen=True)
class StateSpaceSpec:
    heads: int
    vdim: int
    state: int
    groups: int
    norm_groups: int
    conv: int


@dataclass(frozen=True)
class KeyValueAttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    conv: int
    scale: float
    softcap: float            # 0: none
    window: int               # 0: every earlier token
    rot: Optional[RotSpec]


@dataclass(frozen=True)
class TimeMixSpec:
    heads: int
    dim: int
    decay_rank: int           # 0 until known


@dataclass(frozen=True)
class JoinedSpec:
    left: KeyValueAttentionSpec
    right: TimeMixSpec
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class HeadDeltaSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass(frozen=True)
class BoundedDenseSpec:
    ff: int
    limit: float


@dataclass(frozen=True)
class FasanexLayer:
    kind: str
    mixer: Any                # StateSpaceSpec | JoinedSpec | HeadDeltaSpec
    mlp: Optional[BoundedDenseSpec]


def _sub(d: Dict[str, Any], key: str, where: str) -> Dict[str, Any]:
    v = d.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: {where} needs '{key}'")
    return v


def _heads(m: Dict[str, Any], where: str, part: str) -> Tuple[int, int]:
    heads, n = _pos_int(m, "heads", where), _pos_int(m, part, where)
    if heads % n:
        raise ConfigError(f"config.json: {where}: {heads} heads are not a multiple of {n} {part}")
    return heads, n


def _mixer(kind: Any, m: Dict[str, Any], where: str):
    w = where + ".mixer"
    if kind == MAMBA2:
        heads, groups = _heads(m, w, "groups")
        spec = StateSpaceSpec(heads, _pos_int(m, "vdim", w), _pos_int(m, "state", w), groups, _pos_int(m, "norm_groups", w), _pos_int(m, "conv", w))
        if heads * spec.vdim % spec.norm_groups:
            raise ConfigError(f"config.json: {w}: {heads * spec.vdim} channels do not divide into {spec.norm_groups} norm_groups")
        return spec
    if kind == PARALLEL:
        a, b, wl, wr = _sub(m, "left", w), _sub(m, "right", w), w + ".left", w + ".right"
        heads, kv = _heads(a, wl, "kv_heads")
        dim = _pos_int(a, "dim", wl)
        if a.get("vdim", dim) != dim:
            raise ConfigError(f"config.json: {wl}: the values are the keys, so vdim {a['vdim']} must be dim {dim}")
        cap = _number(a, "softcap", wl) if a.get("softcap") is not None else 0.0
        if cap < 0:
            raise ConfigError(f"config.json: {wl}.softcap must be positive (or 0, null or absent for none)")
        window = _pos_int(_sub(a, "mask", wl), "size", wl + ".mask") if a.get("mask") is not None else 0
        left = KeyValueAttentionSpec(heads, kv, dim, _pos_int(a, "conv", wl), _number(a, "scale", wl), cap, window, _rot(a, dim, wl))
        rank = b.get("decay_rank")
        right = TimeMixSpec(_pos_int(b, "heads", wr), _pos_int(b, "dim", wr), int(rank) if rank else 0)
        return JoinedSpec(left, right, _number(m, "left_scale", w), _number(m, "right_scale", w))
    if kind == DELTA:
        heads, kv = _heads(m, w, "kv_heads")
        return HeadDeltaSpec(heads, kv, _pos_int(m, "dim", w), _pos_int(m, "vdim", w), _pos_int(m, "conv", w))
    raise ConfigError(f"config.json: {where}.type '{kind}' is none of '{MAMBA2}', '{PARALLEL}', '{DELTA}'")


@dataclass(frozen=True)
class FasanexConfig(ModelConfig):
    layers: Tuple[FasanexLayer, ...] = ()
    norm_eps: float = 1e-6
    embedding_scale: float = 1.0

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "FasanexConfig":
        vocab, width = _pos_int(raw, "vocab", "config"), _pos_int(raw, "width", "config")
        eps = _number(_sub(raw, "norm", "config"), "eps", "norm")
        if eps <= 0:
            raise ConfigError("config.json: norm.eps must be positive")
        emb = raw.get("embedding")
        scale = _number(emb, "scale", "embedding") if isinstance(emb, dict) and emb.get("scale") is not None else 1.0
        entries = raw.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json: 'layers' must list the layers")
        layers = []
        for i, L in enumerate(entries):
            where = f"layers[{i}]"
            if not isinstance(L, dict) or not isinstance(L.get("mixer"), dict):
                raise ConfigError(f"config.json: {where} needs 'type' and 'mixer'")
            f, mlp = L.get("mlp"), None
            if f is not None:
                if not isinstance(f, dict) or f.get("kind") != "dense":
                    raise ConfigError(f"config.json: {where}.mlp must be null or of kind 'dense' with 'ff' and 'limit'")
                mlp = BoundedDenseSpec(_pos_int(f, "ff", where + ".mlp"), _number(f, "limit", where + ".mlp"))
                if mlp.limit <= 0:
                    raise ConfigError(f"config.json: {where}.mlp.limit must be positive")
            layers.append(FasanexLayer(L.get("type"), _mixer(L.get("type"), L["mixer"], where), mlp))
        max_pos = raw.get("max_positions")
        return cls(architecture=NAME, vocab_size=vocab, hidden_size=width, num_hidden_layers=len(layers),
                   max_position_embeddings=int(max_pos) if max_pos else 1 << 17, bos_token_id=None,
                   eos_token_ids=tuple(int(e) for e in raw.get("eos", ())), layers=tuple(layers), norm_eps=eps, embedding_scale=scale)

    def with_tensor_shapes(self, shapes: Dict[str, Tuple[int, ...]]) -> "FasanexConfig":
        """The sizes that only the checkpoint tells: the rank of each time mixing's decay projection, from its first matrix."""
        layers = list(self.layers)
        for i, L in enumerate(layers):
            if isinstance(L.mixer, JoinedSpec):
                w1 = shapes.get(f"l{i}.mix.right.w1")
                if w1 is None or len(w1) != 2:
                    raise ConfigError(f"layer {i}: the checkpoint has no l{i}.mix.right.w1 to size the decay's projection by")
                layers[i] = replace(L, mixer=replace(L.mixer, right=replace(L.mixer.right, decay_rank=int(w1[0]))))
        return replace(self, layers=tuple(layers))

    def to_json_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"architecture": NAME, "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.norm_eps},
                               "embedding": {"scale": self.embedding_scale}, "max_positions": self.max_position_embeddings, "layers": []}
        if self.eos_token_ids:
            out["eos"] = list(self.eos_token_ids)
        for L in self.layers:
            m = L.mixer
            if isinstance(m, StateSpaceSpec):
                mixer: Dict[str, Any] = {"heads": m.heads, "vdim": m.vdim, "state": m.state, "groups": m.groups, "norm_groups": m.norm_groups,
                                         "conv": m.conv}
            elif isinstance(m, JoinedSpec):
                a, b = m.left, m.right
                left: Dict[str, Any] = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.dim, "conv": a.conv, "scale": a.scale}
                if a.softcap:
                    left["softcap"] = a.softcap
                if a.window:
                    left["mask"] = {"size": a.window}
                if a.rot is not None:
                    left["rot"] = {"dims": a.rot.dims, "base": a.rot.base}
                    if a.rot.scaling is not None:
                        s = a.rot.scaling
                        left["rot"]["scaling"] = {"factor": s.factor, "original": s.original, "fast": s.fast, "slow": s.slow}
                right: Dict[str, Any] = {"heads": b.heads, "dim": b.dim}
                if b.decay_rank:
                    right["decay_rank"] = b.decay_rank
                mixer = {"left": left, "right": right, "left_scale": m.left_scale, "right_scale": m.right_scale}
            else:
                mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.conv}
            mlp = {"kind": "dense", "ff": L.mlp.ff, "limit": L.mlp.limit} if L.mlp is not None else None
            out["layers"].append({"type": L.kind, "mixer": mixer, "mlp": mlp})
        return out
