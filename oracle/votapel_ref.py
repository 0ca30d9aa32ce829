"""Plain CPU implementation of the Votapel decoder, one function per mechanism, for the tests only.

Written from the design's equations with numpy (float64, or any dtype the weights come in).  It shares no code with the
product path: no cache, no sorting of tokens by expert, no batching; a sequence is always computed from its first token.

`cfg` is the normalised configuration (see rai_b200.configs.votapel_config): vocab_size, hidden_size, norm_eps,
residual_mult and `layers`, each {"mixer": {...}, "mlp": {...} or None}; `w` maps the checkpoint's tensor names to arrays.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rms_norm_one_plus(x, w, eps):
    """RMS norm over the last axis whose weight is stored as its difference from one."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * (1.0 + w)


def embed(w, tokens):
    """Token vector plus the learned vector of the position."""
    tokens = np.asarray(tokens, dtype=np.int64)
    return w["embed"][tokens] + w["pos"][:len(tokens)]


def query_temperature(p: int, coef: float, every: int) -> float:
    """Grows with the logarithm of how many whole stretches of `every` positions lie behind position p."""
    return 1.0 + coef * math.log((p + 1) // every + 1)


def soft_cap(s, cap: float):
    return s if not cap else cap * np.tanh(s / cap)


def sink_softmax(s, sink: float):
    """Weights of the scores s; exp(sink) joins the denominator and nothing else."""
    top = max(float(s.max()), sink)
    p = np.exp(s - top)
    return p / (p.sum() + math.exp(sink - top))


def attention(q, k, v, scale, cap, sink, first: int = 0):
    """q [T, H, d] at positions first, first + 1, ...; k [n, G, d], v [n, G, e] from position 0."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]), dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        for i in range(T):
            n = first + i + 1
            s = soft_cap((k[:n, g] @ q[i, h]) * scale, cap)
            out[i, h] = sink_softmax(s, float(sink[h])) @ v[:n, g]
    return out


def attention_mixer(h, w, p, mix):
    """h [T, width] -> [T, width]; the values are the keys."""
    H, G, d = mix["heads"], mix["kv_heads"], mix["dim"]
    T = h.shape[0]
    q = (h @ w[p + ".q"].T + w[p + ".q.b"]).reshape(T, H, d)
    k = (h @ w[p + ".k"].T + w[p + ".k.b"]).reshape(T, G, d)
    if mix["temp_coef"]:
        q = q * np.array([query_temperature(i, mix["temp_coef"], mix["temp_every"]) for i in range(T)]).reshape(T, 1, 1)
    o = attention(q, k, k, mix["scale"], mix["softcap"], w[p + ".sink"])
    return o.reshape(T, H * d) @ w[p + ".o"].T


def glu(h, w, p):
    return (silu(h @ w[p + ".gate"].T) * (h @ w[p + ".up"].T)) @ w[p + ".down"].T


def chosen_experts(scores, top: int, groups: int, keep: int) -> List[int]:
    """Scores [experts] of one token -> the experts it uses.  Of `groups` runs of neighbours the `keep` with the largest
    sum of their two best scores stay; the `top` best experts among those are taken."""
    n = len(scores) // groups
    strength = [sum(sorted(scores[g * n:(g + 1) * n])[-2:]) for g in range(groups)]
    kept = sorted(range(groups), key=lambda g: -strength[g])[:keep]
    open_ = [e for e in range(len(scores)) if e // n in kept]
    return sorted(open_, key=lambda e: -scores[e])[:top]


def moe(h, w, p, mlp):
    """h [T, width]: the chosen experts' outputs weighted by their (not renormalised) scores, plus the shared expert."""
    s = sigmoid(h @ w[p + ".router"].T)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e in chosen_experts(s[t], mlp["top"], mlp["groups"], mlp["keep"]):
            out[t] += s[t, e] * mlp["router_scale"] * glu(h[t], w, f"{p}.e{e}")
    return out + glu(h, w, p + ".shared") if mlp["shared_ff"] else out


def residual_streams(cfg: dict, w: Dict[str, np.ndarray], tokens) -> List[np.ndarray]:
    """The residual stream [T, width] after every layer; both sublayers of a layer read the same normalised input."""
    x = embed(w, tokens)
    out = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}"
        h = rms_norm_one_plus(x, w[p + ".norm1"], cfg["norm_eps"])
        y = attention_mixer(h, w, p + ".mix", layer["mixer"])
        if layer["mlp"] is not None:
            y = y + moe(h, w, p + ".mlp", layer["mlp"])
        x = x + cfg["residual_mult"] * y
        out.append(x)
    return out


def logits(cfg: dict, w: Dict[str, np.ndarray], tokens, streams: Optional[list] = None) -> np.ndarray:
    """[T, vocab] for one sequence computed from its first token."""
    x = (streams or residual_streams(cfg, w, tokens))[-1]
    return rms_norm_one_plus(x, w["final.norm"], cfg["norm_eps"]) @ w["head"].T


def as_float64(w: Dict[str, np.ndarray]) -> Dict[str, np.ndarray]:
    return {k: np.asarray(v, dtype=np.float64) for k, v in w.items()}
