"""A plain statement of the Tuganex decoder in numpy float64: one function per mechanism, whole sequences at once, no
cache.  It shares nothing with the engine: it reads the checkpoint itself and takes the configuration as the dictionary
that config.json holds.

Notation: x is the residual stream [T, width] of ONE request, positions are 0 .. T-1, weights are [out, in] and applied
as x @ W.T.
"""
from __future__ import annotations

import json
import math
import struct

import numpy as np


def read_checkpoint(path):
    """name -> float64 array (integer tables stay integers) of a safetensors file."""
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        head = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, rec in head.items():
        if name == "__metadata__":
            continue
        a, b = rec["data_offsets"]
        raw = data[a:b]
        if rec["dtype"] == "BF16":
            u = np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16
            arr = u.view(np.float32).astype(np.float64)
        elif rec["dtype"] == "F32":
            arr = np.frombuffer(raw, dtype="<f4").astype(np.float64)
        elif rec["dtype"] == "I32":
            arr = np.frombuffer(raw, dtype="<i4").astype(np.int64)
        else:
            raise ValueError(rec["dtype"])
        out[name] = arr.reshape(rec["shape"])
    return out


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def unit_rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def softmax_rows(s):
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


# ---------------------------------------------------------------- positions

def rotate_half(v, pos, dims, base):
    """v [T, ..., d]: dimension i of the first ``dims`` turns with i + dims/2 by pos * base^(-2i/dims)."""
    half = dims // 2
    ang = pos.astype(np.float64)[:, None] * base ** (-2.0 * np.arange(half) / dims)[None, :]
    shape = (v.shape[0],) + (1,) * (v.ndim - 2) + (half,)
    c, s = np.cos(ang).reshape(shape), np.sin(ang).reshape(shape)
    out = v.copy()
    a, b = v[..., :half], v[..., half:dims]
    out[..., :half] = a * c - b * s
    out[..., half:dims] = b * c + a * s
    return out


# ---------------------------------------------------------------- mixers

def retention_scan(q, k, v, decay):
    """S_t = decay S_{t-1} + k_t v_t^T, o_t = S_t^T q_t per head; q, k [T, H, d], v [T, H, dv], decay [H]."""
    T, H, d = q.shape
    S = np.zeros((H, d, v.shape[2]))
    o = np.empty(v.shape)
    for t in range(T):
        S = S * decay[:, None, None] + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hdv,hd->hv", S, q[t])
    return o


def mix_retention(h, w, p, m, eps):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    pos = np.arange(T)
    q = (h @ w[p + "q"].T).reshape(T, H, d)
    k = (h @ w[p + "k"].T).reshape(T, H, d)
    v = (h @ w[p + "v"].T).reshape(T, H, dv)
    rot = m.get("rot")
    if rot:
        q = rotate_half(q, pos, rot["dims"], rot["base"])
        k = rotate_half(k, pos, rot["dims"], rot["base"])
    o = unit_rms(retention_scan(q, k * d ** -0.5, v, np.asarray(m["decay"], dtype=np.float64)), eps)
    return (o.reshape(T, H * dv) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def keys_values(h, w, p, m, eps):
    """Keys [T, G, 2 (maps), d], normed and turned, and values [T, G, dv]."""
    T = h.shape[0]
    G, d, dv = m["kv_heads"], m["dim"], m["vdim"]
    k = rms_norm((h @ w[p + "k"].T).reshape(T, G, 2, d), w[p + "k.norm"], eps)
    if m.get("rot"):
        k = rotate_half(k, np.arange(T), m["rot"]["dims"], m["rot"]["base"])
    return k, (h @ w[p + "v"].T).reshape(T, G, dv)


def lam(w, p, diff):
    return math.exp(float(np.sum(w[p + "lq1"] * w[p + "lk1"]))) - math.exp(float(np.sum(w[p + "lq2"] * w[p + "lk2"]))) + diff


def two_maps(q, k, v, scale):
    """The causal softmax attention of every map: q [T, H, 2, d], k [T, G, 2, d], v [T, G, dv] -> [T, H, 2, dv]."""
    T, H = q.shape[:2]
    per = H // k.shape[1]
    pos = np.arange(T)
    seen = pos[:, None] >= pos[None, :]
    out = np.empty((T, H, 2, v.shape[2]))
    for n in range(H):
        for i in range(2):
            s = np.where(seen, q[:, n, i] @ k[:, n // per, i].T * scale, -np.inf)
            out[:, n, i] = softmax_rows(s) @ v[:, n // per]
    return out


def combine_maps(a, lam_value, diff, eps):
    """[T, H, 2, dv] -> [T, H, dv]."""
    return unit_rms(a[:, :, 0] - lam_value * a[:, :, 1], eps) * (1.0 - diff)


def mix_attention(h, w, p, m, eps, kv):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = rms_norm((h @ w[p + "q"].T).reshape(T, H, 2, d), w[p + "q.norm"], eps)
    if m.get("rot"):
        q = rotate_half(q, np.arange(T), m["rot"]["dims"], m["rot"]["base"])
    o = combine_maps(two_maps(q, kv[0], kv[1], m["scale"]), lam(w, p, m["diff"]), m["diff"], eps)
    return o.reshape(T, H * dv) @ w[p + "o"].T


# ---------------------------------------------------------------- feed-forward

def xielu(z, p, q):
    neg = np.minimum(z, 0.0)
    return np.where(z > 0, softplus(p) * z * z, (0.5 + softplus(q)) * (np.expm1(neg) - neg)) + 0.5 * z


def ff_dense(h, w, p):
    z = h @ w[p + "up"].T + w[p + "up.b"]
    return xielu(z, w[p + "act"][0], w[p + "act"][1]) @ w[p + "down"].T + w[p + "down.b"]


MARGINS = None      # a list, while a caller wants to know how close the routers' calls were: (token, margin) of every call


def _margin(sorted_desc, kept):
    """Per row: the gap between the last value that is kept and the best that is not (inf where all are kept)."""
    if kept >= sorted_desc.shape[-1]:
        return np.full(sorted_desc.shape[0], np.inf)
    with np.errstate(invalid="ignore"):
        gap = sorted_desc[:, kept - 1] - sorted_desc[:, kept]
    return np.where(np.isnan(gap), np.inf, gap)        # -inf minus -inf: closed experts on both sides


def route(h, w, p, r):
    """Chosen outputs [T, top] (experts first, identity experts behind them) and their weights."""
    z = h @ w[p + "router"].T
    n = z.shape[1]
    s = softmax_rows(z)
    choice = s + w[p + "correction"]
    g = r.get("groups")
    margin = np.full(h.shape[0], np.inf)
    if g and g["count"] > 1:
        per = n // g["count"]
        best = choice.reshape(-1, g["count"], per).max(axis=-1)
        keep = np.argsort(-best, axis=-1, kind="stable")[:, :g["keep"]]
        margin = np.minimum(margin, _margin(-np.sort(-best, axis=-1), g["keep"]))
        allowed = np.zeros(best.shape, dtype=bool)
        np.put_along_axis(allowed, keep, True, axis=-1)
        choice = np.where(np.repeat(allowed, per, axis=-1), choice, -np.inf)
    ids = np.argsort(-choice, axis=-1, kind="stable")[:, :r["top"]]
    if MARGINS is not None:
        margin = np.minimum(margin, _margin(-np.sort(-choice, axis=-1), r["top"]))
        MARGINS.extend(enumerate(margin))
    return ids, np.take_along_axis(s, ids, axis=-1)


def expert(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def ff_moe(h, w, p, f):
    ids, ws = route(h, w, p, f["router"])
    E = f["router"]["experts"]
    out = np.zeros_like(h)
    for e in range(E):
        t, c = np.nonzero(ids == e)
        if t.size:
            q = p + f"e{e}."
            out[t] += ws[t, c][:, None] * expert(h[t], w[q + "gate"], w[q + "up"], w[q + "down"])
    out += np.where(ids >= E, ws, 0.0).sum(axis=-1, keepdims=True) * h
    if f.get("shared"):
        q = p + "shared."
        out += sigmoid(h @ w[q + "sg"].T) * expert(h, w[q + "gate"], w[q + "up"], w[q + "down"])
    return out


# ---------------------------------------------------------------- the model

def forward(tokens, w, cfg, streams=None):
    """Logits [T, vocab] of one request given whole; ``streams`` collects x after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens, dtype=np.int64)]
    kept = {}
    for i, L in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", L["mixer"], L.get("mlp")
        if L["type"] == "retention":
            y = mix_retention(x, w, p + "mix.", m, eps)
        else:
            j = m.get("kv_from")
            if j is None:
                kept[i] = keys_values(x, w, p + "mix.", m, eps)
            y = mix_attention(x, w, p + "mix.", m, eps, kept[i if j is None else j])
        x = x + rms_norm(y, w[p + "norm1"], eps)
        if f:
            y = ff_dense(x, w, p + "mlp.") if f["kind"] == "dense" else ff_moe(x, w, p + "mlp.", f)
            x = x + rms_norm(y, w[p + "norm2"], eps)
        if streams is not None:
            streams.append(x.copy())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
