"""Plain CPU implementation of the Malasun decoder, one function per mechanism, for the tests only.

Written from the design's equations with numpy in float64 (or any dtype the weights come in), one token and one head at
a time where that is the clearest form.  It shares no code with the product path: no cache, no chunks, no batching; a
sequence is always computed from its first token.

`cfg` is the normalised configuration (see rai_b200.configs.malasun_config): vocab_size, hidden_size, norm_eps and
`layers`, each {"mixer": {...}, "mlp": {...} or None}; `w` maps the checkpoint's tensor names to arrays.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.log1p(np.exp(-np.abs(z))) + np.maximum(z, 0.0)


def rms_normalise(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def scalar_rms_norm(x, g, eps):
    """The RMS norm whose weight is one number for the whole row."""
    return rms_normalise(x, eps) * float(np.asarray(g).reshape(()))


def xielu(z, pq):
    """z/2 plus a curve: a z^2 for positive z, b (expm1(z) - z) otherwise."""
    p, q = (float(v) for v in np.asarray(pq).reshape(2))
    up = softplus(np.float64(p)) * z * z + 0.5 * z
    zn = np.minimum(z, 0.0)
    down = (0.5 + softplus(np.float64(q))) * (np.expm1(zn) - zn) + 0.5 * z
    return np.where(z > 0, up, down)


def causal_conv(u, taps):
    """u [T, C], taps [C, n]: the last tap weighs the current token, the one before it the previous token, and so on."""
    n = taps.shape[1]
    y = np.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(n):
            s = t - n + 1 + j
            if s >= 0:
                y[t] += taps[:, j] * u[s]
    return y


def alibi_slopes(heads: int):
    return np.array([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)])


def window_attention(q, k, v, scale, slopes, window):
    """q [T, H, d], k [T, G, d], v [T, G, e]: row i sees the `window` keys up to its own; the score loses slope times the distance."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]), dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        for i in range(T):
            lo = max(0, i - window + 1)
            dist = i - np.arange(lo, i + 1)
            s = (k[lo:i + 1, g] @ q[i, h]) * scale - slopes[h] * dist
            p = np.exp(s - s.max())
            out[i, h] = (p / p.sum()) @ v[lo:i + 1, g]
    return out


def gated_linear_recurrence(q, f, v, state=None):
    """One head.  q, f [T, d], v [T, e]: row r of the state keeps f[r] of itself and takes in 1 - f[r] of v; q reads it."""
    S = np.zeros((q.shape[1], v.shape[1]), dtype=q.dtype) if state is None else state.copy()
    o = np.zeros((q.shape[0], v.shape[1]), dtype=q.dtype)
    for t in range(q.shape[0]):
        S = f[t][:, None] * S + (1.0 - f[t])[:, None] * v[t][None, :]
        o[t] = S.T @ q[t]
    return o, S


def hgrn2_mixer(h, w, p, mix, eps):
    """h [T, width] -> [T, width]."""
    H, d, e = mix["heads"], mix["dim"], mix["vdim"]
    T = h.shape[0]
    q = silu(h @ w[p + ".q"].T).reshape(T, H, d)
    lower = w[p + ".lower"]
    f = (lower + (1.0 - lower) * sigmoid(h @ w[p + ".f"].T + w[p + ".f.b"])).reshape(T, H, d)
    v = (h @ w[p + ".v"].T).reshape(T, H, e)
    o = np.zeros((T, H, e), dtype=h.dtype)
    for n in range(H):
        o[:, n], _ = gated_linear_recurrence(q[:, n], f[:, n], v[:, n])
    o = rms_normalise(o, eps) * w[p + ".norm"]
    return o.reshape(T, H * e) @ w[p + ".o"].T


def project_conv(h, w, name, norm_eps: Optional[float]):
    """Projection with its bias, causal convolution, and (queries and keys) the norm over all rows at once."""
    u = causal_conv(h @ w[name].T + w[name + ".b"], w[name + ".conv"])
    return u if norm_eps is None else rms_normalise(u, norm_eps) * w[name + ".norm"]


def attention_mixer(h, w, p, mix, eps, kv):
    """h [T, width] -> ([T, width], (k, v)); kv is another layer's (k, v) when this layer has none of its own."""
    H, G, d, e = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    T = h.shape[0]
    q = project_conv(h, w, p + ".q", eps).reshape(T, H, d)
    if kv is None:
        kv = (project_conv(h, w, p + ".k", eps).reshape(T, G, d), project_conv(h, w, p + ".v", None).reshape(T, G, e))
    o = window_attention(q, kv[0], kv[1], mix["scale"], alibi_slopes(H), mix["window"]).reshape(T, H * e)
    return (o * sigmoid(h @ w[p + ".g"].T)) @ w[p + ".o"].T, kv


def mlp(h, w, p):
    return xielu(h @ w[p + ".up"].T, w[p + ".act"]) @ w[p + ".down"].T


def residual_streams(cfg: dict, w: Dict[str, np.ndarray], tokens) -> List[np.ndarray]:
    """The residual stream [T, width] after every layer."""
    eps = cfg["norm_eps"]
    x = w["embed"][np.asarray(tokens, dtype=np.int64)]
    out, kvs = [], {}
    for i, layer in enumerate(cfg["layers"]):
        mix, p = layer["mixer"], f"l{i}"
        if mix["type"] == "hgrn2":
            y = hgrn2_mixer(x, w, p + ".mix", mix, eps)
        else:
            src = mix.get("kv_from")
            y, kvs[i] = attention_mixer(x, w, p + ".mix", mix, eps, None if src is None else kvs[src])
        x = x + scalar_rms_norm(y, w[p + ".norm1"], eps)
        if layer["mlp"] is not None:
            x = x + scalar_rms_norm(mlp(x, w, p + ".mlp"), w[p + ".norm2"], eps)
        out.append(x)
    return out


def logits(cfg: dict, w: Dict[str, np.ndarray], tokens) -> np.ndarray:
    """[T, vocab] for one sequence computed from its first token."""
    x = residual_streams(cfg, w, tokens)[-1]
    return scalar_rms_norm(x, w["final.norm"], cfg["norm_eps"]) @ w["head"].T


def as_float64(w: Dict[str, np.ndarray]) -> Dict[str, np.ndarray]:
    return {k: np.asarray(v, dtype=np.float64) for k, v in w.items()}
