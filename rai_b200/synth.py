"""Parameter names/shapes of the four decoders and seeded synthetic weights and prompts.

Names follow the derive rule of rai-core/src/nn.rs:256-269 (field path joined by '.', Vec index as
'.i') with the `#[param(rename = ...)]` attributes of qwen2.rs:276-282, phi2.rs:307-313,
phi3.rs:260-266 and gemma.rs:309-318, i.e. the keys of a Hugging Face safetensors checkpoint.

Synthetic weights stand in for real checkpoints (none are available offline): every Linear and
Embedding matrix ~ N(0, 0.02), biases ~ N(0, 0.02), norm weights 1 + N(0, 0.05) (0 + N(0, 0.05) for
gemma, whose norm applies 1 + w; the noise keeps a kernel that forgets the weight from passing), LayerNorm
biases ~ N(0, 0.02); token ids uniform on [0, vocab).
"""
from __future__ import annotations

from typing import Dict, Iterator, List, Tuple

import numpy as np

from . import configs


def param_shapes(cfg: dict) -> List[Tuple[str, Tuple[int, ...], str]]:
    """[(name, shape, kind)] in checkpoint order; kind is 'matrix', 'bias', 'norm_w' or 'norm_b'."""
    a = cfg["arch"]
    if a == "malasun":
        return _malasun_shapes(cfg)
    if a == "votapel":
        return _votapel_shapes(cfg)
    if a == "kufulix":
        return _kufulix_shapes(cfg)
    if a == "fizadra":
        return _fizadra_shapes(cfg)
    H, I, V = cfg["hidden_size"], cfg["intermediate_size"], cfg["vocab_size"]
    nq = cfg["num_attention_heads"]
    nkv = cfg.get("num_key_value_heads") or nq
    d = configs.head_dim(cfg)
    out: List[Tuple[str, Tuple[int, ...], str]] = [("model.embed_tokens.weight", (V, H), "matrix")]
    for i in range(cfg["num_hidden_layers"]):
        p = f"model.layers.{i}."
        if a == "phi3":
            out.append((p + "self_attn.qkv_proj.weight", ((nq + 2 * nkv) * d, H), "matrix"))
            out.append((p + "self_attn.o_proj.weight", (H, nq * d), "matrix"))
            out.append((p + "mlp.gate_up_proj.weight", (2 * I, H), "matrix"))
            out.append((p + "mlp.down_proj.weight", (H, I), "matrix"))
        else:
            bias = a in ("qwen2", "phi2")
            for n, rows in (("q_proj", nq * d), ("k_proj", nkv * d), ("v_proj", nkv * d)):
                out.append((p + f"self_attn.{n}.weight", (rows, H), "matrix"))
                if bias:
                    out.append((p + f"self_attn.{n}.bias", (rows,), "bias"))
            if a == "phi2":
                out.append((p + "self_attn.dense.weight", (H, nq * d), "matrix"))
                out.append((p + "self_attn.dense.bias", (H,), "bias"))
                out.append((p + "mlp.fc1.weight", (I, H), "matrix"))
                out.append((p + "mlp.fc1.bias", (I,), "bias"))
                out.append((p + "mlp.fc2.weight", (H, I), "matrix"))
                out.append((p + "mlp.fc2.bias", (H,), "bias"))
            else:
                out.append((p + "self_attn.o_proj.weight", (H, nq * d), "matrix"))
                out.append((p + "mlp.gate_proj.weight", (I, H), "matrix"))
                out.append((p + "mlp.up_proj.weight", (I, H), "matrix"))
                out.append((p + "mlp.down_proj.weight", (H, I), "matrix"))
        out.append((p + "input_layernorm.weight", (H,), "norm_w"))
        if a == "phi2":
            out.append((p + "input_layernorm.bias", (H,), "norm_b"))
        else:
            out.append((p + "post_attention_layernorm.weight", (H,), "norm_w"))
    if a == "phi2":
        out.append(("model.final_layernorm.weight", (H,), "norm_w"))
        out.append(("model.final_layernorm.bias", (H,), "norm_b"))
    else:
        out.append(("model.norm.weight", (H,), "norm_w"))
    if not configs.tied(cfg):
        out.append(("lm_head.weight", (V, H), "matrix"))
        if a == "phi2":
            out.append(("lm_head.bias", (V,), "bias"))
    return out


def _malasun_shapes(cfg: dict) -> List[Tuple[str, Tuple[int, ...], str]]:
    """Kinds beside the usual ones: 'fan_in' (a matrix that keeps its input's scale), 'gain' (one number), 'conv', 'lower'
    (lower bounds of forget gates, in [0, 1)), 'forget_b' (their biases) and 'act' (the activation's two numbers)."""
    W, V = cfg["hidden_size"], cfg["vocab_size"]
    out: List[Tuple[str, Tuple[int, ...], str]] = [("embed", (V, W), "embed")]
    for i, layer in enumerate(cfg["layers"]):
        mix, mlp, p = layer["mixer"], layer["mlp"], f"l{i}."
        H, d, e = mix["heads"], mix["dim"], mix["vdim"]
        out.append((p + "norm1", (), "gain"))
        if mlp:
            out.append((p + "norm2", (), "gain"))
        m = p + "mix."
        if mix["type"] == "hgrn2":
            out += [(m + "q", (H * d, W), "fan_in"), (m + "f", (H * d, W), "fan_in"), (m + "f.b", (H * d,), "forget_b"),
                    (m + "lower", (H * d,), "lower"), (m + "v", (H * e, W), "fan_in"), (m + "norm", (e,), "norm_w")]
        else:
            parts = [("q", H * d)] + ([] if mix["kv_from"] is not None else [("k", mix["kv_heads"] * d), ("v", mix["kv_heads"] * e)])
            for n, rows in parts:
                out += [(m + n, (rows, W), "fan_in"), (m + n + ".b", (rows,), "bias"), (m + n + ".conv", (rows, mix["conv"]), "conv")]
                if n != "v":
                    out.append((m + n + ".norm", (rows,), "norm_w"))
            out.append((m + "g", (H * e, W), "fan_in"))
        out.append((m + "o", (W, H * e), "fan_in"))
        if mlp:
            out += [(p + "mlp.up", (mlp["ff"], W), "fan_in"), (p + "mlp.down", (W, mlp["ff"]), "fan_in"), (p + "mlp.act", (2,), "act")]
    return out + [("final.norm", (), "gain"), ("head", (V, W), "fan_in")]


def _votapel_shapes(cfg: dict) -> List[Tuple[str, Tuple[int, ...], str]]:
    """Kinds as in _malasun_shapes; 'delta' is a norm weight stored as its difference from one, 'sink' a score."""
    W, V = cfg["hidden_size"], cfg["vocab_size"]
    out: List[Tuple[str, Tuple[int, ...], str]] = [("embed", (V, W), "embed"), ("pos", (cfg["max_positions"], W), "embed")]
    for i, layer in enumerate(cfg["layers"]):
        mix, mlp, p = layer["mixer"], layer["mlp"], f"l{i}."
        q, k = mix["heads"] * mix["dim"], mix["kv_heads"] * mix["dim"]
        out += [(p + "norm1", (W,), "delta"), (p + "mix.q", (q, W), "fan_in"), (p + "mix.q.b", (q,), "bias"),
                (p + "mix.k", (k, W), "fan_in"), (p + "mix.k.b", (k,), "bias"), (p + "mix.sink", (mix["heads"],), "sink"),
                (p + "mix.o", (W, q), "fan_in")]
        if not mlp:
            continue
        parts = [(f"e{e}", mlp["ff"]) for e in range(mlp["experts"])] + ([("shared", mlp["shared_ff"])] if mlp["shared_ff"] else [])
        for name, ff in parts:
            m = f"{p}mlp.{name}."
            out += [(m + "gate", (ff, W), "fan_in"), (m + "up", (ff, W), "fan_in"), (m + "down", (W, ff), "fan_in")]
        out.append((p + "mlp.router", (mlp["experts"], W), "fan_in"))
    return out + [("final.norm", (W,), "delta"), ("head", (V, W), "fan_in")]


def _kufulix_shapes(cfg: dict) -> List[Tuple[str, Tuple[int, ...], str]]:
    """Kinds as in _votapel_shapes; 'step_b' are the biases of a recurrence's step sizes, 'decay' the logarithms of its decay
    rates, 'skip' its direct paths, 'correction' what a router's choice adds to its scores."""
    W, V = cfg["hidden_size"], cfg["vocab_size"]
    out: List[Tuple[str, Tuple[int, ...], str]] = [("embed", (V, W), "embed"), ("embed.norm", (W,), "delta")]
    for i, layer in enumerate(cfg["layers"]):
        mix, mlp, ssd, p = layer["mixer"], layer["mlp"], layer["mixer"]["ssd"], f"l{i}."
        if layer["weights_of"] is not None:
            continue
        out.append((p + "norm1", (W,), "delta"))
        if mlp:
            out.append((p + "norm2", (W,), "delta"))
        m = p + ("mix.left." if ssd else "mix.")
        for n, rows in (("q", mix["heads"] * mix["dim"]), ("k", mix["kv_heads"] * mix["dim"]), ("v", mix["kv_heads"] * mix["vdim"])):
            out += [(m + n, (rows, W), "fan_in"), (m + n + ".b", (rows,), "bias")]
        if mix["qk_norm"]:
            out += [(m + "q.norm", (mix["dim"],), "norm_w"), (m + "k.norm", (mix["dim"],), "norm_w")]
        if mix["head_gate"]:
            out.append((m + "g", (mix["heads"], W), "fan_in"))
        out.append((m + "o", (W, mix["heads"] * mix["vdim"]), "fan_in"))
        if ssd:
            m, h, inner, bc = p + "mix.right.", ssd["heads"], ssd["heads"] * ssd["vdim"], ssd["groups"] * ssd["state"]
            out += [(m + "in", (2 * inner + 2 * bc + h, W), "fan_in"), (m + "conv", (inner + 2 * bc, ssd["conv"]), "conv"),
                    (m + "conv.b", (inner + 2 * bc,), "bias"), (m + "dt_bias", (h,), "step_b"), (m + "A_log", (h,), "decay"),
                    (m + "D", (h,), "skip"), (m + "norm", (inner,), "norm_w"), (m + "o", (W, inner), "fan_in")]
        if mlp:
            m = p + "mlp."
            for e in range(mlp["experts"]):
                out += [(f"{m}e{e}.up", (mlp["ff"], W), "fan_in"), (f"{m}e{e}.down", (W, mlp["ff"]), "fan_in")]
            out += [(m + "router", (mlp["experts"] + mlp["identity"], W), "fan_in"),
                    (m + "correction", (mlp["experts"] + mlp["identity"],), "correction")]
    return out + [("final.norm", (W,), "delta"), ("head", (V, W), "fan_in")]


def _fizadra_shapes(cfg: dict) -> List[Tuple[str, Tuple[int, ...], str]]:
    """Kinds as in _votapel_shapes; 'talk' is how heads mix their scores, 'depth' a layer's weights of everything before it."""
    W, V = cfg["hidden_size"], cfg["vocab_size"]
    out: List[Tuple[str, Tuple[int, ...], str]] = [("embed", (V, W), "embed")]
    for i, layer in enumerate(cfg["layers"]):
        mix, mlp, p = layer["mixer"], layer["mlp"], f"l{i}."
        H, d, e, m = mix["heads"], mix["dim"], mix["vdim"], f"l{i}.mix."
        out += [(p + n, (W,), "norm_w") for n in (("norm1", "norm2", "norm1b", "norm2b") if mlp else ("norm1", "norm1b"))]
        if mix["type"] == "latent_attention":
            out += [(m + "dq", (mix["q_rank"], W), "fan_in"), (m + "dq.norm", (mix["q_rank"],), "norm_w"),
                    (m + "uq", (H * (d + mix["rot_dim"]), mix["q_rank"]), "fan_in")]
            if mix["kv_from"] is None:
                out += [(m + "dkv", (mix["kv_rank"] + mix["rot_dim"], W), "fan_in"), (m + "dkv.norm", (mix["kv_rank"],), "norm_w")]
            out += [(m + "uk", (H * d, mix["kv_rank"]), "fan_in"), (m + "uv", (H * e, mix["kv_rank"]), "fan_in")]
            if mix["sink"]:
                out.append((m + "sink", (H,), "sink"))
            out.append((m + "g", (H * e if mix["gate"] == "elements" else H, W), "fan_in"))
        else:
            for n, rows in (("q", H * d), ("k", mix["kv_heads"] * d), ("v", mix["kv_heads"] * e)):
                out += [(m + n, (rows, W), "fan_in"), (m + n + ".b", (rows,), "bias")]
            out += [(m + "q.norm", (d,), "norm_w"), (m + "k.norm", (d,), "norm_w"), (m + "talk", (H, H), "talk")]
        out.append((m + "o", (W, H * e), "fan_in"))
        if mlp:
            out += [(p + "mlp.up", (mlp["ff"], W), "fan_in"), (p + "mlp.down", (W, mlp["ff"]), "fan_in")]
        out.append((p + "dwa", (i + 2,), "depth"))
    return out + [("final.norm", (W,), "norm_w"), ("head", (V, W), "fan_in")]


def bf16_round(x: np.ndarray) -> np.ndarray:
    """float32 -> nearest-even bfloat16 -> float32 (so the CPU oracle and the GPU see the same values)."""
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32)
    r = ((u >> 16) & 1) + np.uint32(0x7FFF)
    return ((u + r) & np.uint32(0xFFFF0000)).view(np.float32)


_DRAWS = {
    "embed": lambda r, s: r.standard_normal(s),
    "fan_in": lambda r, s: r.standard_normal(s) / np.sqrt(s[1]),
    "gain": lambda r, s: 1.0 + 0.2 * r.standard_normal(s),
    "conv": lambda r, s: r.standard_normal(s) / np.sqrt(s[1]),
    "lower": lambda r, s: r.uniform(0.0, 0.9, s),
    "forget_b": lambda r, s: r.uniform(0.0, 6.0, s),
    "delta": lambda r, s: 0.2 * r.standard_normal(s),
    "sink": lambda r, s: r.standard_normal(s),
    "act": lambda r, s: r.uniform(-1.0, 1.0, s),
    "step_b": lambda r, s: r.uniform(-5.0, 0.0, s),
    "decay": lambda r, s: r.uniform(-1.0, 2.5, s),
    "skip": lambda r, s: 1.0 + 0.3 * r.standard_normal(s),
    "correction": lambda r, s: 0.05 * r.standard_normal(s),
    "talk": lambda r, s: np.eye(s[0]) + r.standard_normal(s) / np.sqrt(s[0]),
    "depth": lambda r, s: np.append(0.3 * r.standard_normal(s[0] - 1), 1.0),
}


def iter_weights(cfg: dict, seed: int, round_bf16: bool = True) -> Iterator[Tuple[str, np.ndarray]]:
    """Yields (name, float32 array) in checkpoint order from numpy PCG64(seed)."""
    rng = np.random.Generator(np.random.PCG64(seed))
    gemma = cfg["arch"] == "gemma"
    for name, shape, kind in param_shapes(cfg):
        if kind in ("matrix", "bias"):
            w = (rng.standard_normal(shape, dtype=np.float32) * np.float32(0.02)).astype(np.float32)
            # norm-like perturbation keeps the test weights from being trivially 1/0 everywhere
        elif kind == "norm_w":
            base = 0.0 if gemma else 1.0
            w = (base + rng.standard_normal(shape, dtype=np.float32) * np.float32(0.05)).astype(np.float32)
        elif kind in _DRAWS:
            w = np.asarray(_DRAWS[kind](rng, shape), dtype=np.float32)
        else:
            w = (rng.standard_normal(shape, dtype=np.float32) * np.float32(0.02)).astype(np.float32)
        yield name, (bf16_round(w) if round_bf16 else w).reshape(shape)


def weights(cfg: dict, seed: int, round_bf16: bool = True) -> Dict[str, np.ndarray]:
    return dict(iter_weights(cfg, seed, round_bf16))


def prompt(cfg: dict, batch: int, seq: int, seed: int) -> np.ndarray:
    """[batch, seq] uint32 token ids, uniform on [0, vocab)."""
    rng = np.random.Generator(np.random.PCG64(seed + 1))
    return rng.integers(0, cfg["vocab_size"], size=(batch, seq), dtype=np.int64).astype(np.uint32)
