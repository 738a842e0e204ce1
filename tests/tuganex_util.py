"""Helpers of the Tuganex tests: small configurations of their own, a writer of random weights whose scale lets every
mechanism matter, and the comparison of the engine with the plain implementation (`plain_tuganex`).  The writer names
every tensor itself, so a weight slot that the engine forgets or misnames shows as a loading error."""
from __future__ import annotations

import functools
import json
import os
from typing import Dict, List, Tuple

import numpy as np

import plain_tuganex as P
from zidivik_util import PartHarness, bf16_round, load_part, write_model  # noqa: F401  (helpers that know no architecture)


def _rot(rot):
    return None if rot is None else {"dims": rot[0], "base": rot[1]}


def attn(heads, kv_heads, dim, vdim, scale, diff, rot=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff, "rot": _rot(rot)}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m}


def retention(heads, dim, vdim, decay, rot=None):
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay), "rot": _rot(rot)}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, identity, top, ff, groups, keep, shared):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top, "groups": {"count": groups, "keep": keep}},
            "shared": {"ff": shared} if shared else None}


def layer(mixer, mlp):
    return dict(mixer, mlp=mlp)


# T1: grouped heads with values wider than a map, part of a map turned; a layer on another's keys with other heads, scale and
# diff; decays from fast to none at all; identity experts that share groups with real ones; a layer without feed-forward.
T1 = {"architecture": "Tuganex", "vocab": 211, "width": 80, "norm": {"eps": 1e-5}, "layers": [
    layer(attn(6, 2, 24, 40, 0.21, 0.3, (16, 100.0)), moe(9, 3, 3, 40, 3, 2, 56)),
    layer(retention(3, 40, 24, (0.75, 0.99, 1.0), (16, 50.0)), None),
    layer(attn(4, 2, 24, 40, 0.35, 0.55, (16, 100.0), kv_from=0), dense(96)),
    layer(retention(2, 16, 48, (0.5, 0.96875), (16, 1000.0)), moe(10, 2, 4, 24, 4, 3, 0)),
]}
# T2: sizes that are no multiples of 8 (the plain kernels in bfloat16 too); a recurrence first; groups of one router output;
# no identity experts in one layer, more of them than experts in another; one value head for five query heads; no rotation.
T2 = {"architecture": "Tuganex", "vocab": 97, "width": 70, "norm": {"eps": 1e-6}, "layers": [
    layer(retention(3, 14, 10, (0.9, 0.3, 0.97), (6, 30.0)), dense(30)),
    layer(attn(5, 1, 10, 14, 0.4, 0.2, (6, 20.0)), moe(6, 0, 2, 22, 6, 3, 18)),
    layer(attn(3, 3, 18, 6, 0.3, 0.8), moe(2, 4, 2, 12, 1, 1, 0)),
    layer(attn(2, 1, 10, 14, 0.6, 0.45, (6, 20.0), kv_from=1), None),
]}
# T3: maps of 64 over values of 128 and recurrent heads of 128 (the tensor-core kernels' sizes); one expert of sixteen, all
# groups kept; a reader with as many heads as key heads.
T3 = {"architecture": "Tuganex", "vocab": 131, "width": 64, "norm": {"eps": 1e-6}, "layers": [
    layer(attn(4, 2, 64, 128, 0.125, 0.35, (64, 10000.0)), moe(16, 0, 1, 48, 4, 4, 32)),
    layer(retention(2, 128, 128, (0.984375, 0.998), (128, 10000.0)), dense(72)),
    layer(attn(2, 2, 64, 128, 0.2, 0.7, (64, 10000.0), kv_from=0), dense(48)),
]}
# T4: no routed experts (a run in bfloat16 cannot route otherwise than the plain one): long requests in reduced precision
T4 = {"architecture": "Tuganex", "vocab": 151, "width": 96, "norm": {"eps": 1e-6}, "layers": [
    layer(attn(4, 2, 16, 48, 0.3, 0.5, (8, 500.0)), dense(128)),
    layer(retention(4, 32, 64, (0.875, 0.96875, 0.9921875, 0.998046875), (32, 500.0)), dense(64)),
    layer(attn(8, 2, 16, 48, 0.25, 0.4, (8, 500.0), kv_from=0), None),
    layer(attn(3, 1, 40, 24, 0.16, 0.25, (24, 2000.0)), dense(80)),
]}
# A token whose query and key are all but orthogonal (|cosine| below 1e-3) makes a first position whose normed output no number
# format determines: o = (q . k) v, divided by its own size.  The seeds below draw no such token.
CONFIGS = {"T1": (T1, 3), "T2": (T2, 10), "T3": (T3, 5), "T4": (T4, 13)}


def tensors_of(cfg: dict, seed: int) -> Dict[str, np.ndarray]:
    """Random float32 tensors for ``cfg``, by name.  Matrices N(0, g / sqrt(in)) so that activations keep their size through the
    layers; norm weights around 1; biases of order 1; corrections that spread the router outputs' chances."""
    rng = np.random.default_rng(seed)
    D, V = cfg["width"], cfg["vocab"]
    W: Dict[str, np.ndarray] = {}

    def mat(name, out, inn, gain=1.0):
        W[name] = (rng.standard_normal((out, inn)) * gain / np.sqrt(inn)).astype(np.float32)

    def vec(name, shape, mean=0.0, std=1.0):
        W[name] = (mean + std * rng.standard_normal(shape)).astype(np.float32)

    W["embed"] = rng.standard_normal((V, D)).astype(np.float32)
    for i, L in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", L["mixer"], L.get("mlp")
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        vec(p + "norm1", D, 0.8, 0.1)
        if L["type"] == "attention":
            G = m["kv_heads"]
            mat(p + "mix.q", H * 2 * d, D)
            if m.get("kv_from") is None:
                mat(p + "mix.k", G * 2 * d, D)
                mat(p + "mix.v", G * dv, D)
                vec(p + "mix.k.norm", d, 1.0, 0.3)
            vec(p + "mix.q.norm", d, 1.0, 0.3)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                vec(p + "mix." + n, d, 0.0, 0.7 / np.sqrt(d) ** 0.5)
            mat(p + "mix.o", D, H * dv)
        else:
            for n, rows in (("q", H * d), ("k", H * d), ("v", H * dv), ("g", H * dv)):
                mat(p + "mix." + n, rows, D, 1.3)
            mat(p + "mix.o", D, H * dv)
        if f is not None:
            vec(p + "norm2", D, 0.8, 0.1)
        if f is not None and f["kind"] == "dense":
            mat(p + "mlp.up", f["ff"], D, 1.5)
            vec(p + "mlp.up.b", f["ff"], 0.0, 0.5)
            mat(p + "mlp.down", D, f["ff"])
            vec(p + "mlp.down.b", D, 0.0, 0.5)
            vec(p + "mlp.act", 2, 0.0, 1.0)
        elif f is not None:
            r = f["router"]
            n = r["experts"] + r["identity"]
            mat(p + "mlp.router", n, D, 1.5)
            vec(p + "mlp.correction", n, 0.0, 0.1)
            for e in range(r["experts"]):
                mat(p + f"mlp.e{e}.gate", f["expert"]["ff"], D, 1.5)
                mat(p + f"mlp.e{e}.up", f["expert"]["ff"], D, 1.5)
                mat(p + f"mlp.e{e}.down", D, f["expert"]["ff"], 2.0)
            if f.get("shared"):
                mat(p + "mlp.shared.gate", f["shared"]["ff"], D, 1.5)
                mat(p + "mlp.shared.up", f["shared"]["ff"], D)
                mat(p + "mlp.shared.down", D, f["shared"]["ff"])
                mat(p + "mlp.shared.sg", 1, D, 1.5)
    vec("final.norm", D, 1.0, 0.1)
    mat("head", V, D)
    return W


@functools.lru_cache(maxsize=None)
def _model(model_dir: str):
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    return cfg, P.read_checkpoint(os.path.join(model_dir, "model.safetensors"))


@functools.lru_cache(maxsize=None)
def _plain(model_dir: str, tokens: Tuple[int, ...]):
    cfg, W = _model(model_dir)
    P.MARGINS = []
    try:
        logits = P.forward(list(tokens), W, cfg)
        close = [t for t, m in P.MARGINS if m < CLOSE_CALL]
    finally:
        P.MARGINS = None
    return logits, (min(close) if close else len(tokens))


def plain_logits(model_dir: str, tokens) -> np.ndarray:
    return _plain(model_dir, tuple(int(t) for t in tokens))[0]


def first_close_call(model_dir: str, tokens) -> int:
    """First position at which some router separates what it keeps (a group, an output) from the best it leaves out by
    less than `CLOSE_CALL`: from there on a run in reduced precision may route otherwise (len(tokens) if none)."""
    return _plain(model_dir, tuple(int(t) for t in tokens))[1]


CLOSE_CALL = 0.01
# |engine - plain| as a fraction of the largest |plain logit| of the request.  float32: sums in another order.  bfloat16:
# operands, activations between products and the cache are rounded to 8 bits of mantissa.  A fault of the cache, a state, a
# mask or a table moves the positions it touches by tenths; the float32 comparison on the same traces allows 2e-5.
TOL = {"float32": 2e-5, "bfloat16": 5e-2}


def compare_with_plain(model_dir_f32: str, reqs: Dict[str, List[int]], got, dtype: str, label: str = "") -> float:
    """Every logits row of a trace against the plain implementation.  In bfloat16, positions from a request's first close
    router call on are left out (the float32 run covers them).  Names the first wrong (request, position)."""
    worst, n = 0.0, 0
    for name, toks in reqs.items():
        ref = plain_logits(model_dir_f32, toks)
        scale = float(np.abs(ref).max())
        upto = len(toks) if dtype == "float32" else first_close_call(model_dir_f32, toks)
        assert set(got[name]) == set(range(len(toks))), f"{label}: {name} misses positions"
        for p in range(upto):
            row = got[name][p]
            assert np.isfinite(row).all(), f"{label}: {name} position {p}: logits are not finite"
            err = float(np.abs(row - ref[p]).max()) / scale
            worst, n = max(worst, err), n + 1
            assert err <= TOL[dtype], (f"{label}: first wrong place: request {name} position {p} of {len(toks)}: "
                                       f"error {err:.3e} of the largest logit, allowed {TOL[dtype]:.1e}")
    print(f"[tuganex] {label}: {n} positions, worst {worst:.3e}")
    return worst


def requests(name: str, lengths, seed: int) -> Dict[str, List[int]]:
    rng = np.random.default_rng(seed)
    vocab = CONFIGS[name][0]["vocab"]
    return {f"r{i}": rng.integers(0, vocab, size=n).tolist() for i, n in enumerate(lengths)}
