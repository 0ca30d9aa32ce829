"""Plain CPU implementation of the Fizadra decoder, one function per mechanism, for the tests only.

Written from the design's equations with numpy (float64, or any dtype the weights come in).  It shares no code with the
product path: no cache, no absorbed projections, no batching; a sequence is always computed from its first token.

`cfg` is the normalised configuration (see rai_b200.configs.fizadra_config): vocab_size, hidden_size, norm_eps, norm_groups and
`layers`, each {"mixer": {...}, "mlp": {...} or None}; `w` maps the checkpoint's tensor names to arrays.
"""
from __future__ import annotations

import math
from typing import Dict, List

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def rms(x, eps):
    """x over the root mean square of its last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def group_norm(x, w, groups, eps):
    """Each of `groups` equal parts of the last axis over its own root mean square, the whole times w."""
    return rms(x.reshape(x.shape[:-1] + (groups, -1)), eps).reshape(x.shape) * w


def depth_average(weights, xs):
    """One weighted sum of the embedding and every layer's result so far."""
    assert len(weights) == len(xs)
    out = np.zeros_like(xs[0])
    for c, x in zip(weights, xs):
        out = out + c * x
    return out


def rotary_frequencies(rot) -> List[float]:
    """One angle per position and pair.  With scaling, pairs below a first index keep their frequency, those above a second one
    have it divided by `factor`, with a linear passage between; the indices are where a pair turns `fast` and `slow` times
    over `original` positions."""
    dims, base, s = rot["dims"], rot["base"], rot.get("scaling")
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if s:
            def index(turns):
                return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
            lo = max(math.floor(index(s["fast"])), 0)
            hi = min(math.ceil(index(s["slow"])), dims - 1)
            ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            f = f / s["factor"] * ramp + f * (1.0 - ramp)
        out.append(f)
    return out


def rotary_amplitude(rot) -> float:
    s = rot.get("scaling")
    return 0.1 * math.log(s["factor"]) + 1.0 if s else 1.0


def rotate(x, rot, first: int = 0):
    """x [T, heads, d] at positions first, first + 1, ...: pairs of neighbours (interleaved) or of the two halves turn; what
    lies beyond rot["dims"] stays."""
    if not rot:
        return x
    dims, a = rot["dims"], rotary_amplitude(rot)
    out = x.copy()
    for t in range(x.shape[0]):
        for i, f in enumerate(rotary_frequencies(rot)):
            c, s = a * math.cos((first + t) * f), a * math.sin((first + t) * f)
            j, k = (2 * i, 2 * i + 1) if rot["interleaved"] else (i, i + dims // 2)
            u, v = x[t, :, j], x[t, :, k]
            out[t, :, j], out[t, :, k] = u * c - v * s, v * c + u * s
    return out


def softmax_with_sink(s, sink=None):
    """Weights of the scores s [n]; exp(sink) joins the denominator (None: nothing does)."""
    top = s.max() if sink is None else max(s.max(), sink)
    e = np.exp(s - top)
    return e / (e.sum() + (0.0 if sink is None else np.exp(sink - top)))


def attention(q, k, v, scale, sink=None, talk=None, first: int = 0):
    """q [T, H, d] at positions first, first + 1, ...; k [n, G, d], v [n, G, e] from position 0.  talk [H, H] mixes the heads'
    scores before the softmax; sink [H]."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]), dtype=q.dtype)
    for i in range(T):
        n = first + i + 1
        s = np.stack([(k[:n, h // (H // G)] @ q[i, h]) * scale for h in range(H)])
        if talk is not None:
            s = talk @ s
        for h in range(H):
            out[i, h] = softmax_with_sink(s[h], None if sink is None else sink[h]) @ v[:n, h // (H // G)]
    return out


def talking_attention_mixer(h, w, p, mix, eps):
    H, G, d, e = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    T = h.shape[0]
    q = rms((h @ w[p + ".q"].T + w[p + ".q.b"]).reshape(T, H, d), eps) * w[p + ".q.norm"]
    k = rms((h @ w[p + ".k"].T + w[p + ".k.b"]).reshape(T, G, d), eps) * w[p + ".k.norm"]
    v = (h @ w[p + ".v"].T + w[p + ".v.b"]).reshape(T, G, e)
    o = attention(rotate(q, mix["rot"]), rotate(k, mix["rot"]), v, mix["scale"], np.zeros(H), w[p + ".talk"])
    return o.reshape(T, -1) @ w[p + ".o"].T


def latent(h, w, p, mix, eps):
    """What a token leaves behind: the normed latent [T, kv_rank] and the turned key part [T, rot_dim] that all heads share."""
    u = h @ w[p + ".dkv"].T
    r = mix["kv_rank"]
    return rms(u[:, :r], eps) * w[p + ".dkv.norm"], rotate(u[:, None, r:], mix["rot"])[:, 0]


def latent_attention_mixer(h, w, p, mix, eps, c, turned):
    """c, turned: this layer's `latent`, or another layer's."""
    H, d, e = mix["heads"], mix["dim"], mix["vdim"]
    T = h.shape[0]
    cq = rms(h @ w[p + ".dq"].T, eps) * w[p + ".dq.norm"]
    q = (cq @ w[p + ".uq"].T).reshape(T, H, d + mix["rot_dim"])
    q = np.concatenate([q[:, :, :d], rotate(q[:, :, d:], mix["rot"])], -1)
    k = np.concatenate([(c @ w[p + ".uk"].T).reshape(T, H, d), np.repeat(turned[:, None], H, 1)], -1)
    o = attention(q, k, (c @ w[p + ".uv"].T).reshape(T, H, e), mix["scale"], w[p + ".sink"] if mix["sink"] else None)
    g = sigmoid(h @ w[p + ".g"].T)
    o = o * (g[:, :, None] if mix["gate"] == "heads" else g.reshape(T, H, e))
    return o.reshape(T, -1) @ w[p + ".o"].T


def feed_forward(h, w, p):
    return np.square(np.maximum(h @ w[p + ".up"].T, 0.0)) @ w[p + ".down"].T


def residual_streams(cfg, w, tokens) -> List[np.ndarray]:
    """The stream after every layer, its depth average included."""
    eps, groups = cfg["norm_eps"], cfg["norm_groups"]
    x = w["embed"][np.asarray(tokens)]
    history, out, latents = [x], [], {}
    for i, layer in enumerate(cfg["layers"]):
        mix, p = layer["mixer"], f"l{i}"
        h = group_norm(x, w[p + ".norm1"], groups, eps)
        if mix["type"] == "latent_attention":
            src = mix["kv_from"]
            if src is None:
                latents[i] = latent(h, w, p + ".mix", mix, eps)
            y = latent_attention_mixer(h, w, p + ".mix", mix, eps, *latents[i if src is None else src])
        else:
            y = talking_attention_mixer(h, w, p + ".mix", mix, eps)
        x = x + group_norm(y, w[p + ".norm1b"], groups, eps)
        if layer["mlp"]:
            y = feed_forward(group_norm(x, w[p + ".norm2"], groups, eps), w, p + ".mlp")
            x = x + group_norm(y, w[p + ".norm2b"], groups, eps)
        history.append(x)
        x = depth_average(w[p + ".dwa"], history)
        out.append(x)
    return out


def logits(cfg, w, tokens) -> np.ndarray:
    x = residual_streams(cfg, w, tokens)[-1]
    return group_norm(x, w["final.norm"], cfg["norm_groups"], cfg["norm_eps"]) @ w["head"].T


def greedy(cfg, w, prompt, steps: int) -> List[int]:
    """The last index among equal maxima, like the sampler."""
    t = [int(v) for v in prompt]
    for _ in range(steps):
        z = logits(cfg, w, t)[-1]
        t.append(int(len(z) - 1 - np.argmax(z[::-1])))
    return t[len(prompt):]


def as_float64(weights: Dict[str, np.ndarray]) -> Dict[str, np.ndarray]:
    return {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}
