"""Typed configuration of the Tuganex decoder, read from its own ``config.json`` keys.

Top level: ``architecture`` (a string), ``vocab``, ``width``, ``norm.eps`` and ``layers``, a list with one entry per
layer: ``type`` (which mixer), ``mixer`` (its sizes and constants) and ``mlp`` (null, ``{"kind": "dense", "ff": n}``, or
``{"kind": "moe", "expert": {"ff": n}, "router": {"experts", "identity", "top", "groups": {"count", "keep"}}, "shared":
{"ff": n} or null}``).

* ``attention``: ``heads``, ``kv_heads``, ``dim`` (of each of a head's two maps), ``vdim``, ``scale``, ``diff``, ``rot``
  (``dims``, ``base``; null: no rotation), ``kv_from`` (the layer whose keys and values it uses; absent: its own).
* ``retention``: ``heads``, ``dim``, ``vdim``, ``decay`` (a number per head), ``rot``.

Every size and constant comes from the file; nothing is assumed equal between layers.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .model_config import ConfigError, ModelConfig
from .zidivik_config import _number, _pos_int

NAME = "Tuganex"

ATTENTION, RETENTION = "attention", "retention"


@dataclass(frozen=True)
class RotSpec:
    dims: int
    base: float


@dataclass(frozen=True)
class DifferentialSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    rot: Optional[RotSpec]
    kv_from: Optional[int]      # the layer whose keys and values this one uses, None for its own


@dataclass(frozen=True)
class RetentionSpec:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    rot: Optional[RotSpec]


@dataclass(frozen=True)
class DenseSpec:
    ff: int


@dataclass(frozen=True)
class MoeSpec:
    ff: int
    experts: int
    identity: int               # router outputs behind the experts whose output is the input itself
    top: int
    groups: int
    keep: int
    shared_ff: int              # 0: no expert that every token takes


@dataclass(frozen=True)
class TuganexLayer:
    kind: str
    mixer: Any                  # DifferentialSpec | RetentionSpec
    mlp: Any                    # None | DenseSpec | MoeSpec


def _obj(raw: Dict[str, Any], key: str, where: str, optional: bool = False) -> Optional[Dict[str, Any]]:
    v = raw.get(key)
    if v is None and optional:
        return None
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: {where}.{key} must be an object")
    return v


def _rot(m: Dict[str, Any], dim: int, where: str) -> Optional[RotSpec]:
    r = _obj(m, "rot", where, optional=True)
    if r is None:
        return None
    w = where + ".rot"
    dims, base = _pos_int(r, "dims", w, allow_zero=True), _number(r, "base", w)
    if dims % 2 or dims > dim:
        raise ConfigError(f"config.json: {w}.dims {dims} must be even and at most dim {dim}")
    if base <= 0:
        raise ConfigError(f"config.json: {w}.base must be positive")
    return RotSpec(dims, base) if dims else None


def _mlp(f: Any, where: str):
    if f is None:
        return None
    if not isinstance(f, dict) or f.get("kind") not in ("dense", "moe"):
        raise ConfigError(f"config.json: {where} must be null or of kind 'dense' or 'moe'")
    if f["kind"] == "dense":
        return DenseSpec(_pos_int(f, "ff", where))
    e, r, w = _obj(f, "expert", where), _obj(f, "router", where), where + ".router"
    experts, top = _pos_int(r, "experts", w), _pos_int(r, "top", w)
    identity = _pos_int(r, "identity", w, allow_zero=True) if r.get("identity") is not None else 0
    g = _obj(r, "groups", w, optional=True)
    groups, keep = (1, 1) if g is None else (_pos_int(g, "count", w + ".groups"), _pos_int(g, "keep", w + ".groups"))
    n = experts + identity
    if n % groups or keep > groups or top > keep * (n // groups):
        raise ConfigError(f"config.json: {w}: {n} router outputs in {groups} groups, {keep} kept, {top} chosen do not fit")
    s = _obj(f, "shared", where, optional=True)
    return MoeSpec(_pos_int(e, "ff", where + ".expert"), experts, identity, top, groups, keep, _pos_int(s, "ff", where + ".shared") if s else 0)


@dataclass(frozen=True)
class TuganexConfig(ModelConfig):
    layers: Tuple[TuganexLayer, ...] = ()
    norm_eps: float = 1e-6

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "TuganexConfig":
        vocab, width = _pos_int(raw, "vocab", "config"), _pos_int(raw, "width", "config")
        eps = _number(_obj(raw, "norm", "config"), "eps", "norm")
        if eps <= 0:
            raise ConfigError("config.json: norm.eps must be positive")
        entries = raw.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json: 'layers' must list the layers")
        layers = []
        for i, L in enumerate(entries):
            where = f"layers[{i}]"
            if not isinstance(L, dict) or not isinstance(L.get("mixer"), dict):
                raise ConfigError(f"config.json: {where} needs 'type' and 'mixer'")
            m, kind, w = L["mixer"], L.get("type"), where + ".mixer"
            if kind == ATTENTION:
                heads, kv, dim = _pos_int(m, "heads", w), _pos_int(m, "kv_heads", w), _pos_int(m, "dim", w)
                if heads % kv:
                    raise ConfigError(f"config.json: {w}: {heads} heads are not a multiple of {kv} kv_heads")
                kv_from = m.get("kv_from")
                mixer: Any = DifferentialSpec(heads, kv, dim, _pos_int(m, "vdim", w), _number(m, "scale", w), _number(m, "diff", w),
                                              _rot(m, dim, w), None if kv_from is None else _pos_int(m, "kv_from", w, allow_zero=True))
                if mixer.kv_from is not None:
                    src = layers[mixer.kv_from].mixer if mixer.kv_from < i else None
                    if not isinstance(src, DifferentialSpec) or src.kv_from is not None or \
                            (src.kv_heads, src.dim, src.vdim) != (kv, dim, mixer.vdim):
                        raise ConfigError(f"config.json: {w}.kv_from {mixer.kv_from} is no earlier attention layer with keys and values of its own "
                                          f"and this layer's kv_heads, dim and vdim")
            elif kind == RETENTION:
                heads, dim, decay = _pos_int(m, "heads", w), _pos_int(m, "dim", w), m.get("decay")
                if not isinstance(decay, list) or len(decay) != heads or \
                        not all(isinstance(x, (int, float)) and not isinstance(x, bool) and 0 <= x <= 1 for x in decay):
                    raise ConfigError(f"config.json: {w}.decay must list {heads} numbers from 0 to 1, one per head")
                mixer = RetentionSpec(heads, dim, _pos_int(m, "vdim", w), tuple(float(x) for x in decay), _rot(m, dim, w))
            else:
                raise ConfigError(f"config.json: {where}.type '{kind}' is neither '{ATTENTION}' nor '{RETENTION}'")
            layers.append(TuganexLayer(kind, mixer, _mlp(L.get("mlp"), where + ".mlp")))
        max_pos = raw.get("max_positions")
        return cls(architecture=NAME, vocab_size=vocab, hidden_size=width, num_hidden_layers=len(layers),
                   max_position_embeddings=int(max_pos) if max_pos else 1 << 17, bos_token_id=None,
                   eos_token_ids=tuple(int(e) for e in raw.get("eos", ())), layers=tuple(layers), norm_eps=eps)

    def to_json_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"architecture": NAME, "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.norm_eps},
                               "max_positions": self.max_position_embeddings, "layers": []}
        if self.eos_token_ids:
            out["eos"] = list(self.eos_token_ids)
        for L in self.layers:
            m = L.mixer
            if isinstance(m, DifferentialSpec):
                mixer: Dict[str, Any] = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "diff": m.diff}
                if m.kv_from is not None:
                    mixer["kv_from"] = m.kv_from
            else:
                mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "decay": list(m.decay)}
            if m.rot is not None:
                mixer["rot"] = {"dims": m.rot.dims, "base": m.rot.base}
            f = L.mlp
            if f is None:
                mlp: Any = None
            elif isinstance(f, DenseSpec):
                mlp = {"kind": "dense", "ff": f.ff}
            else:
                mlp = {"kind": "moe", "expert": {"ff": f.ff},
                       "router": {"experts": f.experts, "identity": f.identity, "top": f.top, "groups": {"count": f.groups, "keep": f.keep}},
                       "shared": {"ff": f.shared_ff} if f.shared_ff else None}
            out["layers"].append({"type": L.kind, "mixer": mixer, "mlp": mlp})
        return out
