"""Plain restatement of the Fasanex decoder, for tests only.

Whole sequences, no cache, no batching, numpy float64 throughout, one function per mechanism.
Nothing here is imported by the engine and nothing of the engine is imported here: the file has
its own reader of config.json and of safetensors.

Notation.  T tokens at positions 0..T-1, width D.  The stream starts as the table's rows times a
constant.  A norm's weight w is kept as its distance from one: the factor is 1 + w.  A layer is

    x <- x + norm1b(mixer(norm1(x)));   x <- x + norm2b(ff(norm2(x)))

(the second half only where a layer has a feed-forward).  Three mixers: `mamba2` (a scalar decay per
head over a shared pair of input and output vectors), `parallel` (windowed softmax attention whose
values are its keys before norm and rotation, beside a recurrence with a decay per key channel that
reads each token blended with the one before it) and `delta` (the gated delta rule with one decay
per head).
"""
from __future__ import annotations

import json
import math
import os
import struct

import numpy as np

F = np.float64


def read_safetensors(path: str) -> dict:
    with open(path, "rb") as f:
        blob = f.read()
    (hlen,) = struct.unpack("<Q", blob[:8])
    header = json.loads(blob[8:8 + hlen].decode("utf-8"))
    base = 8 + hlen
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        b, e = info["data_offsets"]
        raw = blob[base + b: base + e]
        dt = info["dtype"]
        if dt == "BF16":
            arr = (np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16).view(np.float32).astype(F)
        elif dt == "F32":
            arr = np.frombuffer(raw, dtype="<f4").astype(F)
        elif dt == "I32":
            arr = np.frombuffer(raw, dtype="<i4")
        else:
            raise ValueError(f"plain reader: dtype {dt} of {name}")
        out[name] = arr.reshape(tuple(info["shape"])).copy()
    return out


def read_model(model_dir: str):
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    return cfg, read_safetensors(os.path.join(model_dir, "model.safetensors"))


# ---- small functions -------------------------------------------------------------------------

def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def stream_norm(x, w, eps):
    """The norm of the model width: its weight is stored as a distance from one."""
    return unit_rms(x, eps) * (1.0 + w)


def linear(x, w):
    """Rows of x times w^T, w stored [out, in]."""
    return x @ w.T


def causal_conv(u, w, b=None):
    """Per channel c: y[t, c] = sum_j w[c, j] u[t - (taps - 1) + j, c] (+ b[c]); nothing lies in front of token 0."""
    T, taps = u.shape[0], w.shape[1]
    y = np.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            n = t - (taps - 1) + j
            if n >= 0:
                y[t] += w[:, j] * u[n]
    return y if b is None else y + b


# ---- rotation --------------------------------------------------------------------------------

def rotary_frequencies(rot: dict):
    """(a frequency per pair of the first rot['dims'] dimensions, the factor on cos and sin).  With a scaling, pair i of
    frequency f_i = base^(-2i/dims) turns with f_i (1 - r_i + r_i / factor), r a ramp from 0 to 1 between the pairs whose
    wavelengths fit `fast` and `slow` times into the original context."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    factor, orig = float(sc["factor"]), float(sc["original"])

    def pair_of(turns):
        return dims * math.log(orig / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(pair_of(float(sc["fast"]))), 0)
    hi = min(math.ceil(pair_of(float(sc["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi * (1.0 - r) + fi / factor * r)
    return np.array(out, dtype=F), 0.1 * math.log(factor) + 1.0


def rotate_half(x: np.ndarray, positions: np.ndarray, freq: np.ndarray, magnitude: float) -> np.ndarray:
    """x [T, heads, d]: dimensions i and i + n (n = len(freq), i < n) turn by positions * freq[i], times the magnitude;
    the rest of a head passes unchanged."""
    out = x.copy()
    n = freq.shape[0]
    ang = positions[:, None].astype(F) * freq[None, :]
    c, s = magnitude * np.cos(ang)[:, None, :], magnitude * np.sin(ang)[:, None, :]
    u, v = x[..., :n], x[..., n:2 * n]
    out[..., :n] = u * c - v * s
    out[..., n:2 * n] = v * c + u * s
    return out


# ---- mixers ----------------------------------------------------------------------------------

def state_space(x, B, C, dt, A_log, D):
    """Per head n with group n // (H / G): S_t = exp(-exp(A_log) dt) S_{t-1} + dt B_t x_t^T, y_t = S_t^T C_t + D x_t.
    x [T, H, P], B, C [T, G, N], dt [T, H]."""
    T, H, P = x.shape
    G, N = B.shape[1:]
    S = np.zeros((H, N, P), dtype=F)
    y = np.zeros((T, H, P), dtype=F)
    for t in range(T):
        for n in range(H):
            g = n // (H // G)
            S[n] = math.exp(-math.exp(A_log[n]) * dt[t, n]) * S[n] + dt[t, n] * np.outer(B[t, g], x[t, n])
            y[t, n] = S[n].T @ C[t, g] + D[n] * x[t, n]
    return y


def grouped_unit_rms(y, groups, eps):
    """y [T, n] in `groups` equal parts, each over its own root mean square."""
    T, n = y.shape
    return unit_rms(y.reshape(T, groups, n // groups), eps).reshape(T, n)


def mamba2_mixer(h, W, p, m, eps):
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    f = linear(h, W[p + "in"])
    z, u, dt = f[:, :inner], f[:, inner:2 * inner + 2 * G * N], f[:, 2 * inner + 2 * G * N:]
    u = silu(causal_conv(u, W[p + "conv"], W[p + "conv.b"]))
    x, B, C = u[:, :inner].reshape(T, H, P), u[:, inner:inner + G * N].reshape(T, G, N), u[:, inner + G * N:].reshape(T, G, N)
    y = state_space(x, B, C, softplus(dt + W[p + "dt_bias"]), W[p + "A_log"], W[p + "D"]).reshape(T, inner)
    y = grouped_unit_rms(y * silu(z), m["norm_groups"], eps) * W[p + "norm"]
    return linear(y, W[p + "o"])


def window_attention(q, k, v, scale, cap, window):
    """Softmax attention, q [T, H, d], k [T, G, d], v [T, G, dv], query head n on key head n // (H / G); token i sees
    0 <= i - j < window; scores scaled, then capped by cap * tanh(s / cap)."""
    T, H, _ = q.shape
    G, dv = k.shape[1], v.shape[2]
    out = np.zeros((T, H, dv), dtype=F)
    for n in range(H):
        g = n // (H // G)
        for i in range(T):
            a = max(0, i - window + 1) if window else 0
            s = (k[a:i + 1, g] @ q[i, n]) * scale
            if cap:
                s = cap * np.tanh(s / cap)
            w = np.exp(s - s.max())
            out[i, n] = (w @ v[a:i + 1, g]) / w.sum()
    return out


def attention_side(h, W, p, m, eps):
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q = causal_conv(linear(h, W[p + "q"]), W[p + "q.conv"]).reshape(T, H, d)
    k = causal_conv(linear(h, W[p + "k"]), W[p + "k.conv"]).reshape(T, G, d)
    v = k                                                    # as it left the convolution
    q, k = unit_rms(q, eps) * W[p + "q.norm"], unit_rms(k, eps) * W[p + "k.norm"]
    if m.get("rot"):
        freq, mag = rotary_frequencies(m["rot"])
        q, k = (rotate_half(a, np.arange(T), freq, mag) for a in (q, k))
    o = window_attention(q, k, v, float(m["scale"]), float(m.get("softcap") or 0.0), int((m.get("mask") or {}).get("size", 0)))
    return linear(o.reshape(T, H * d) * sigmoid(linear(h, W[p + "g"])), W[p + "o"])


def bonus_recurrence(r, k, v, w, u):
    """Per head o_t = (S_{t-1} + diag(u) k_t v_t^T)^T r_t, S_t = diag(w_t) S_{t-1} + k_t v_t^T.  All [T, H, d], u [H, d]."""
    T, H, d = r.shape
    S = np.zeros((H, d, d), dtype=F)
    out = np.zeros((T, H, d), dtype=F)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S + u[:, :, None] * kv, r[t])
        S = w[t][:, :, None] * S + kv
    return out


def time_mix_side(h, W, p, m, eps):
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    before = np.concatenate([np.zeros((1, h.shape[1])), h[:-1]])

    def mix(s):
        return h + (before - h) * W[p + "mu." + s]
    r, k, v = (linear(mix(s), W[p + s]).reshape(T, H, d) for s in "rkv")
    gate = silu(linear(mix("g"), W[p + "g"]))
    w = np.exp(-np.exp(linear(np.tanh(linear(mix("w"), W[p + "w1"])), W[p + "w2"]) + W[p + "w0"])).reshape(T, H, d)
    o = bonus_recurrence(r, k, v, w, W[p + "u"])
    return linear(unit_rms(o, eps).reshape(T, H * d) * W[p + "norm"] * gate, W[p + "o"])


def parallel_mixer(h, W, p, m, eps):
    return float(m["left_scale"]) * attention_side(h, W, p + "left.", m["left"], eps) + \
        float(m["right_scale"]) * time_mix_side(h, W, p + "right.", m["right"], eps)


def delta_rule(q, k, v, beta, g):
    """Per value head n with key head n // (H / G): S <- g S; S <- S + k (beta (v - S^T k))^T; o = S^T q.
    q, k [T, G, d], v [T, H, dv], beta, g [T, H]."""
    T, H, dv = v.shape
    G, d = q.shape[1:]
    S = np.zeros((H, d, dv), dtype=F)
    out = np.zeros((T, H, dv), dtype=F)
    for t in range(T):
        for n in range(H):
            a = n // (H // G)
            S[n] *= g[t, n]
            S[n] += np.outer(k[t, a], beta[t, n] * (v[t, n] - S[n].T @ k[t, a]))
            out[t, n] = S[n].T @ q[t, a]
    return out


def unit_vectors(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def delta_mixer(h, W, p, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(linear(h, W[p + n]), W[p + n + ".conv"])) for n in "qkv")
    q = unit_vectors(q.reshape(T, G, d)) / math.sqrt(d)
    k = unit_vectors(k.reshape(T, G, d))
    g = np.exp(-np.exp(W[p + "A_log"]) * softplus(linear(h, W[p + "a"]) + W[p + "dt_bias"]))
    o = delta_rule(q, k, v.reshape(T, H, dv), sigmoid(linear(h, W[p + "b"])), g)
    o = unit_rms(o, eps) * W[p + "norm"]
    return linear(o.reshape(T, H * dv) * silu(linear(h, W[p + "g"])), W[p + "o"])


def clamped_ff(h, W, p, m):
    """g = min(W_gate h, limit), u = W_up h bounded on both sides; W_down (g sigmoid(1.702 g) (u + 1))."""
    lim = float(m["limit"])
    g, u = np.minimum(linear(h, W[p + "gate"]), lim), np.clip(linear(h, W[p + "up"]), -lim, lim)
    return linear(g * sigmoid(1.702 * g) * (u + 1.0), W[p + "down"])


MIXERS = {"mamba2": mamba2_mixer, "parallel": parallel_mixer, "delta": delta_mixer}


# ---- the model -------------------------------------------------------------------------------

def layer_forward(x, W, cfg, i):
    L, p, eps = cfg["layers"][i], f"l{i}.", float(cfg["norm"]["eps"])
    y = MIXERS[L["type"]](stream_norm(x, W[p + "norm1"], eps), W, p + "mix.", L["mixer"], eps)
    x = x + stream_norm(y, W[p + "norm1b"], eps)
    if L.get("mlp") is not None:
        z = clamped_ff(stream_norm(x, W[p + "norm2"], eps), W, p + "mlp.", L["mlp"])
        x = x + stream_norm(z, W[p + "norm2b"], eps)
    return x


def forward(cfg: dict, W: dict, tokens, layers_out=None) -> np.ndarray:
    """Logits [T, vocab] of one sequence; ``layers_out``, a list, receives x after every layer."""
    x = W["embed"][np.asarray(tokens)] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    for i in range(len(cfg["layers"])):
        x = layer_forward(x, W, cfg, i)
        if layers_out is not None:
            layers_out.append(x.copy())
    return linear(stream_norm(x, W["final.norm"], float(cfg["norm"]["eps"])), W["head"])
