"""Helpers of the Fasanex tests: small configurations of their own, a writer of random weights whose scale lets every mechanism
matter, and the comparison of the engine with the plain implementation (`plain_fasanex`).  The writer names every tensor itself, so a
weight slot that the engine forgets or misnames shows as a loading error."""
from __future__ import annotations

import functools
from typing import Dict, List, Tuple

import numpy as np

import plain_fasanex as P
from zidivik_util import PartHarness, bf16_round, load_part, write_model  # noqa: F401  (helpers that know no architecture)


def rot(dims, base, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def mamba2(heads, vdim, state, groups, norm_groups, conv):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}}


def parallel(heads, kv_heads, dim, conv, scale, cap, window, rotary, r_heads, r_dim, rank, scales=(0.7, 1.2)):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "conv": conv, "scale": scale}
    if cap:
        left["softcap"] = cap
    if window:
        left["mask"] = {"size": window}
    if rotary:
        left["rot"] = rotary
    return {"type": "parallel", "mixer": {"left": left, "right": {"heads": r_heads, "dim": r_dim, "decay_rank": rank},
                                          "left_scale": scales[0], "right_scale": scales[1]}}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def layer(mixer, ff=None, limit=1.0):
    return dict(mixer, mlp={"kind": "dense", "ff": ff, "limit": limit} if ff else None)


# F1: the parallel layer first; three different windows would not fit one model, so two of them, one shorter than a page; part of a
# head rotated with all parts of the ramp; state sizes that differ from value sizes both ways; two layers without feed-forward.
F1 = {"architecture": "Fasanex", "vocab": 151, "width": 72, "norm": {"eps": 1e-5}, "embedding": {"scale": 3.5}, "layers": [
    layer(parallel(6, 2, 24, 3, 0.35, 8.0, 21, rot(16, 100.0, (4.0, 64, 8.0, 0.5)), 2, 24, 9), 80, 0.8),
    layer(mamba2(6, 16, 24, 3, 2, 4), None),
    layer(delta(4, 2, 16, 24, 2), 48, 1.5),
    layer(parallel(4, 4, 32, 2, 0.2, 20.0, 9, rot(32, 1000.0), 3, 16, 5, (1.1, 0.6)), None),
    layer(mamba2(4, 40, 8, 1, 4, 2), 56, 2.0),
]}
# F2: sizes that are no multiples of 8 or 4; one key head in several places; no window, no rotation, no cap in one layer; one filter tap;
# one norm part; five taps.
F2 = {"architecture": "Fasanex", "vocab": 89, "width": 70, "norm": {"eps": 1e-6}, "layers": [
    layer(mamba2(3, 10, 14, 1, 1, 1), 30, 1.0),
    layer(parallel(5, 1, 18, 5, 0.4, 0.0, 0, None, 3, 14, 3), 44, 0.5),
    layer(delta(5, 1, 22, 18, 3), None),
    layer(parallel(2, 2, 10, 1, 0.5, 5.0, 33, rot(6, 50.0, (8.0, 32, 4.0, 1.0)), 5, 6, 7), 62, 3.0),
    layer(delta(3, 1, 26, 30, 5), 34, 1.0),
]}
# F3: the sizes of the tensor-core paths - heads of 128 (portions on the tcgen05 kernel), states of 64 and 128 - behind a window of
# more than a chunk.
F3 = {"architecture": "Fasanex", "vocab": 131, "width": 64, "norm": {"eps": 1e-6}, "embedding": {"scale": 0.5}, "layers": [
    layer(mamba2(4, 64, 128, 2, 2, 4), 72, 1.2),
    layer(parallel(4, 2, 128, 4, 0.09, 15.0, 100, rot(128, 10000.0, (8.0, 128, 16.0, 1.0)), 2, 64, 16, (0.9, 1.3)), None),
    layer(delta(4, 2, 128, 64, 4), 48, 1.0),
    layer(delta(2, 1, 64, 128, 4), None),
]}
CONFIGS = {"F1": (F1, 3), "F2": (F2, 8), "F3": (F3, 5)}


def tensors_of(cfg: dict, seed: int) -> Dict[str, np.ndarray]:
    """Random float32 tensors for ``cfg``, by name.  Matrices N(0, g / sqrt(in)) so that activations keep their size through the layers;
    the width's norm weights around 0, the others around 1; decays from fast to slow."""
    rng = np.random.default_rng(seed)
    D, V = cfg["width"], cfg["vocab"]
    W: Dict[str, np.ndarray] = {}

    def mat(name, out, inn, gain=1.0):
        W[name] = (rng.standard_normal((out, inn)) * gain / np.sqrt(inn)).astype(np.float32)

    def vec(name, n, mean=0.0, std=1.0):
        W[name] = (mean + std * rng.standard_normal(n)).astype(np.float32)

    def conv(name, channels, taps):
        w = rng.standard_normal((channels, taps)) * 0.5
        w[:, -1] += 0.7
        W[name] = w.astype(np.float32)

    W["embed"] = rng.standard_normal((V, D)).astype(np.float32)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        q = p + "mix."
        for n in ("norm1", "norm1b"):
            vec(p + n, D, 0.0, 0.2)
        if L["type"] == "mamba2":
            inner, gn = m["heads"] * m["vdim"], m["groups"] * m["state"]
            mat(q + "in", 2 * inner + 2 * gn + m["heads"], D, 1.5)
            conv(q + "conv", inner + 2 * gn, m["conv"])
            vec(q + "conv.b", inner + 2 * gn, 0.0, 0.3)
            vec(q + "dt_bias", m["heads"], -1.5, 1.0)
            vec(q + "A_log", m["heads"], -0.5, 1.0)
            vec(q + "D", m["heads"], 0.5, 0.5)
            vec(q + "norm", inner, 1.0, 0.2)
            mat(q + "o", D, inner)
        elif L["type"] == "parallel":
            a, b = m["left"], m["right"]
            H, G, d = a["heads"], a["kv_heads"], a["dim"]
            for n, rows in (("q", H * d), ("k", G * d)):
                mat(q + "left." + n, rows, D, 1.5)
                conv(q + f"left.{n}.conv", rows, a["conv"])
                vec(q + f"left.{n}.norm", d, 1.2, 0.3)
            mat(q + "left.g", H * d, D, 1.5)
            mat(q + "left.o", D, H * d)
            n, r = b["heads"] * b["dim"], b["decay_rank"]
            for s in "rkvgw":
                W[q + "right.mu." + s] = rng.uniform(0.0, 1.0, D).astype(np.float32)
            for s in "rkvg":
                mat(q + "right." + s, n, D, 1.5)
            mat(q + "right.w1", r, D, 1.5)
            mat(q + "right.w2", n, r, 1.5)
            vec(q + "right.w0", n, -2.5, 1.5)
            vec(q + "right.u", n, 0.5, 0.7)
            W[q + "right.u"] = W[q + "right.u"].reshape(b["heads"], b["dim"])
            vec(q + "right.norm", n, 1.0, 0.2)
            mat(q + "right.o", D, n)
        else:
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for n, rows in (("q", G * d), ("k", G * d), ("v", H * dv)):
                mat(q + n, rows, D, 1.5)
                conv(q + n + ".conv", rows, m["conv"])
            for n in ("a", "b"):
                mat(q + n, H, D, 1.5)
            mat(q + "g", H * dv, D, 1.5)
            vec(q + "A_log", H, -1.0, 1.0)
            vec(q + "dt_bias", H, -1.0, 1.0)
            vec(q + "norm", dv, 1.0, 0.2)
            mat(q + "o", D, H * dv)
        f = L.get("mlp")
        if f is not None:
            for n in ("norm2", "norm2b"):
                vec(p + n, D, 0.0, 0.2)
            mat(p + "mlp.gate", f["ff"], D, 1.5)
            mat(p + "mlp.up", f["ff"], D, 1.5)
            mat(p + "mlp.down", D, f["ff"])
    vec("final.norm", D, 0.0, 0.2)
    mat("head", V, D)
    return W


@functools.lru_cache(maxsize=None)
def _model(model_dir: str):
    return P.read_model(model_dir)


@functools.lru_cache(maxsize=None)
def plain_logits(model_dir: str, tokens: Tuple[int, ...]) -> np.ndarray:
    cfg, W = _model(model_dir)
    return P.forward(cfg, W, list(tokens))


# |engine - plain| as a fraction of the largest |plain logit| of the request: the most at any one position, and the most for the mean
# over a trace's positions.  Every sublayer's result is normed to unit size before it is added, so a small result's rounding enters the
# stream at full weight: in bfloat16 single positions reach a few hundredths while the mean stays near one hundredth.  A fault of the
# cache, a state or a mask moves the positions it touches by tenths and more, and the float32 comparison allows 2e-5.
TOL = {"float32": 2e-5, "bfloat16": 8e-2}
TOL_MEAN = {"float32": 2e-5, "bfloat16": 1.6e-2}


def compare_with_plain(model_dir_f32: str, reqs: Dict[str, List[int]], got, dtype: str, label: str = "") -> float:
    """Every logits row of a trace against the plain implementation; names the first wrong (request, position)."""
    worst, errs = 0.0, []
    for name, toks in reqs.items():
        ref = plain_logits(model_dir_f32, tuple(toks))
        scale = float(np.abs(ref).max())
        assert set(got[name]) == set(range(len(toks))), f"{label}: {name} misses positions"
        for p in range(len(toks)):
            row = got[name][p]
            assert np.isfinite(row).all(), f"{label}: {name} position {p}: logits are not finite"
            err = float(np.abs(row - ref[p]).max()) / scale
            worst = max(worst, err)
            errs.append(err)
            assert err <= TOL[dtype], (f"{label}: first wrong place: request {name} position {p} of {len(toks)}: "
                                       f"error {err:.3e} of the largest logit, allowed {TOL[dtype]:.1e}")
    mean = float(np.mean(errs))
    print(f"[fasanex] {label}: {len(errs)} positions, worst {worst:.3e}, mean {mean:.3e}")
    assert mean <= TOL_MEAN[dtype], f"{label}: mean error {mean:.3e} over {len(errs)} positions, allowed {TOL_MEAN[dtype]:.1e}"
    return worst


def steady_first_tokens(cfg: dict, W: Dict[str, np.ndarray], floor: float = 0.05) -> List[int]:
    """Tokens that may open a request in a comparison at reduced precision.  At a request's first token the read-outs of the delta rule
    and of time mixing are (q . k) v and (r . (u k)) v, and the norm over the head keeps of the factor only its sign: where it is tiny
    beside the vectors' lengths, rounding decides the sign, in any implementation.  This lists the tokens for which no head's is."""
    eps = float(cfg["norm"]["eps"])
    Wd = {n: a.astype(np.float64) for n, a in W.items()}

    def clear(a, b):
        return bool((np.abs((a * b).sum(-1)) >= floor * np.linalg.norm(a, axis=-1) * np.linalg.norm(b, axis=-1)).all())
    good = []
    for tok in range(int(cfg["vocab"])):
        x, ok = Wd["embed"][[tok]] * float((cfg.get("embedding") or {}).get("scale", 1.0)), True
        for i, L in enumerate(cfg["layers"]):
            m, p = L["mixer"], f"l{i}.mix."
            h = P.stream_norm(x, Wd[f"l{i}.norm1"], eps)
            if L["type"] == "delta":
                q, k = (P.silu(P.causal_conv(P.linear(h, Wd[p + n]), Wd[p + n + ".conv"])).reshape(m["kv_heads"], m["dim"]) for n in "qk")
                ok = ok and clear(q, k)
            elif L["type"] == "parallel":
                b = m["right"]
                r, k = (P.linear(h - h * Wd[p + "right.mu." + s], Wd[p + "right." + s]).reshape(b["heads"], b["dim"]) for s in "rk")
                ok = ok and clear(r, Wd[p + "right.u"] * k)
            x = P.layer_forward(x, Wd, cfg, i)
        if ok:
            good.append(tok)
    return good


@functools.lru_cache(maxsize=None)
def _steady_of(name: str) -> Tuple[int, ...]:
    cfg, seed = CONFIGS[name]
    return tuple(steady_first_tokens(cfg, bf16_round(tensors_of(cfg, seed))))


def requests(name: str, lengths, seed: int) -> Dict[str, List[int]]:
    """Random requests r0, r1, ... for the configuration ``name``, each opened by a token of `steady_first_tokens`."""
    cfg = CONFIGS[name][0]
    rng = np.random.default_rng(seed)
    good = _steady_of(name)
    assert len(good) >= 8, f"{name}: only {len(good)} tokens can open a request"
    out = {}
    for i, n in enumerate(lengths):
        toks = rng.integers(0, cfg["vocab"], size=n).tolist()
        toks[0] = int(good[int(rng.integers(0, len(good)))])
        out[f"r{i}"] = toks
    return out
