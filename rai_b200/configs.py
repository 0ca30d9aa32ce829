"""Decoder configurations.

Malasun, Votapel, Kufulix and Fizadra, designs described layer by layer (no counterpart in the reference), have configurations
of their own shape: see `malasun_config`, `votapel_config`, `kufulix_config` and `fizadra_config`.  For the others, field names
follow the reference `Config` structs (rai-models/src/llm/qwen2.rs:8-24, phi2.rs:9-24, phi3.rs:9-24, gemma.rs:12-27) as they
appear in a Hugging Face config.json, plus `arch`.
`BASELINE` holds the five benchmark configurations; `TINY` holds small models of the same four
architectures for parity tests.
"""
from __future__ import annotations

import copy
import ctypes
import json
import os
from typing import Dict

from . import _lib

ARCH_IDS = {"qwen2": _lib.ARCH_QWEN2, "phi2": _lib.ARCH_PHI2, "phi3": _lib.ARCH_PHI3, "gemma": _lib.ARCH_GEMMA,
            "malasun": _lib.ARCH_MALASUN, "votapel": _lib.ARCH_VOTAPEL, "kufulix": _lib.ARCH_KUFULIX,
            "fizadra": _lib.ARCH_FIZADRA}
LAYERED = ("malasun", "votapel", "kufulix", "fizadra")   # described layer by layer: rb_model_create_layers
MIXER_IDS = {"attention": _lib.MIXER_ATTENTION, "hgrn2": _lib.MIXER_HGRN2, "attention_ssd": _lib.MIXER_ATTENTION_SSD,
             "latent_attention": _lib.MIXER_LATENT}
# serde names of rai-nn/src/activations.rs:5-17
ACT_IDS = {"silu": _lib.ACT_SILU, "gelu_new": _lib.ACT_GELU_TANH, "newgelu": _lib.ACT_GELU_TANH,
           "gelu": _lib.ACT_GELU_ERF, "relu": _lib.ACT_RELU}

BASELINE: Dict[str, dict] = {
    # C1: Qwen2-0.5B architecture; batch 1, 128-token prompt, 128 greedy steps
    "qwen2-0.5b": dict(arch="qwen2", vocab_size=151936, hidden_size=896, intermediate_size=4864, num_hidden_layers=24,
                       num_attention_heads=14, num_key_value_heads=2, max_position_embeddings=4096,
                       sliding_window=32768, rope_theta=1e6, rms_norm_eps=1e-6, hidden_act="silu",
                       tie_word_embeddings=True),
    # C2: Phi-2 architecture; batch 8, 512-token prompts, 256 greedy steps
    "phi2": dict(arch="phi2", vocab_size=51200, hidden_size=2560, intermediate_size=10240, num_hidden_layers=32,
                 num_attention_heads=32, num_key_value_heads=32, max_position_embeddings=2048, rope_theta=1e4,
                 layer_norm_eps=1e-5, hidden_act="gelu_new", partial_rotary_factor=0.4, qk_layernorm=False,
                 tie_word_embeddings=False),
    # C3: Phi-3-mini architecture; batch 4 x 2048-token prompts, 64 decode steps
    "phi3-mini": dict(arch="phi3", vocab_size=32064, hidden_size=3072, intermediate_size=8192, num_hidden_layers=32,
                      num_attention_heads=32, num_key_value_heads=32, max_position_embeddings=4096, rope_theta=1e4,
                      rms_norm_eps=1e-5, hidden_act="silu"),
    # C4: Gemma-2B architecture; batch 32 decode from a 1024-token cache, 128 greedy steps
    "gemma-2b": dict(arch="gemma", vocab_size=256000, hidden_size=2048, intermediate_size=16384, num_hidden_layers=18,
                     num_attention_heads=8, num_key_value_heads=1, head_dim=256, max_position_embeddings=8192,
                     rope_theta=1e4, rms_norm_eps=1e-6, hidden_act="gelu_new", attention_bias=False),
    # C5: Qwen2-7B architecture; prefill 8 x 4096, then batch-64 decode at 2048-token context, 256 steps
    "qwen2-7b": dict(arch="qwen2", vocab_size=152064, hidden_size=3584, intermediate_size=18944, num_hidden_layers=28,
                     num_attention_heads=28, num_key_value_heads=4, max_position_embeddings=8192, sliding_window=131072,
                     rope_theta=1e6, rms_norm_eps=1e-6, hidden_act="silu", tie_word_embeddings=False),
}

TINY: Dict[str, dict] = {
    "tiny-qwen2": dict(arch="qwen2", vocab_size=512, hidden_size=256, intermediate_size=320, num_hidden_layers=2,
                  num_attention_heads=4, num_key_value_heads=2, max_position_embeddings=256, sliding_window=4096,
                  rope_theta=1e6, rms_norm_eps=1e-6, hidden_act="silu", tie_word_embeddings=False),
    "tiny-qwen2-tied": dict(arch="qwen2", vocab_size=384, hidden_size=128, intermediate_size=192, num_hidden_layers=2,
                       num_attention_heads=2, num_key_value_heads=2, max_position_embeddings=256, sliding_window=4096,
                       rope_theta=1e6, rms_norm_eps=1e-6, hidden_act="silu", tie_word_embeddings=True),
    # 7 query heads per KV head and head_dim 128, the grouping of the 7B benchmark configuration
    "tiny-qwen2-g7": dict(arch="qwen2", vocab_size=640, hidden_size=896, intermediate_size=768, num_hidden_layers=2,
                     num_attention_heads=7, num_key_value_heads=1, max_position_embeddings=512, sliding_window=4096,
                     rope_theta=1e6, rms_norm_eps=1e-6, hidden_act="silu", tie_word_embeddings=False),
    # narrow shapes: K = 40 and 64 (less than one 64-wide K slice), N = 40, a 64-row vocabulary
    "tiny-qwen2-narrow": dict(arch="qwen2", vocab_size=64, hidden_size=128, intermediate_size=40, num_hidden_layers=2,
                              num_attention_heads=2, num_key_value_heads=2, max_position_embeddings=256,
                              sliding_window=4096, rope_theta=1e6, rms_norm_eps=1e-6, hidden_act="silu",
                              tie_word_embeddings=False),
    # the head layout of the 7B benchmark configuration (28 query heads over 4 KV heads) at small width
    "tiny-qwen2-28h": dict(arch="qwen2", vocab_size=1024, hidden_size=1792, intermediate_size=1024, num_hidden_layers=2,
                           num_attention_heads=28, num_key_value_heads=4, max_position_embeddings=256,
                           sliding_window=4096, rope_theta=1e6, rms_norm_eps=1e-6, hidden_act="silu",
                           tie_word_embeddings=False),
    "tiny-phi2": dict(arch="phi2", vocab_size=320, hidden_size=160, intermediate_size=640, num_hidden_layers=2,
                 num_attention_heads=2, num_key_value_heads=2, max_position_embeddings=256, rope_theta=1e4,
                 layer_norm_eps=1e-5, hidden_act="gelu_new", partial_rotary_factor=0.4, qk_layernorm=False,
                 tie_word_embeddings=False),
    "tiny-phi3": dict(arch="phi3", vocab_size=448, hidden_size=192, intermediate_size=512, num_hidden_layers=2,
                 num_attention_heads=2, num_key_value_heads=2, max_position_embeddings=256, rope_theta=1e4,
                 rms_norm_eps=1e-5, hidden_act="silu"),
    "tiny-gemma": dict(arch="gemma", vocab_size=640, hidden_size=512, intermediate_size=1024, num_hidden_layers=2,
                  num_attention_heads=2, num_key_value_heads=1, head_dim=256, max_position_embeddings=256,
                  rope_theta=1e4, rms_norm_eps=1e-6, hidden_act="gelu_new", attention_bias=False),
}


def malasun_layer(kind: str, heads: int, dim: int, vdim: int, mlp: int = 0, kv_heads: int = 0, conv: int = 1, window: int = 0,
                  scale: float = 0.0, kv_from=None) -> dict:
    """One entry of a Malasun configuration's `layers`; mlp = 0 leaves the feed-forward out."""
    mixer = dict(type=kind, heads=heads, dim=dim, vdim=vdim)
    if kind == "attention":
        mixer.update(kv_heads=kv_heads or heads, conv=conv, window=window, scale=scale or dim ** -0.5, kv_from=kv_from)
    return dict(mixer=mixer, mlp=dict(kind="dense", ff=mlp) if mlp else None)


def _malasun(vocab: int, width: int, layers, eps: float = 1e-6) -> dict:
    return dict(arch="malasun", vocab_size=vocab, hidden_size=width, norm_eps=eps, layers=layers)


def _malasun_bench(vocab: int, width: int, heads: int, kv_heads: int, ff: int, pairs: int, window: int) -> dict:
    """Alternating hgrn2 and attention layers of 128-wide heads, each with a feed-forward."""
    layers = []
    for _ in range(pairs):
        layers.append(malasun_layer("hgrn2", heads, 128, 128, ff))
        layers.append(malasun_layer("attention", heads, 128, 128, ff, kv_heads, 4, window))
    return _malasun(vocab, width, layers)


MALASUN: Dict[str, dict] = {
    # sizes that resemble a real model's layers, for throughput measurements (random weights)
    "malasun-1k": _malasun_bench(32000, 1024, 8, 2, 4096, 8, 1024),
    "malasun-2k": _malasun_bench(32000, 2048, 16, 4, 8192, 6, 1024),
    "malasun-4k": _malasun_bench(32000, 4096, 32, 8, 16384, 3, 1024),
    # small models for tests
    "tiny-malasun": _malasun(320, 160, [
        malasun_layer("attention", 4, 40, 32, 200, 2, 4, 21), malasun_layer("hgrn2", 3, 32, 48, 0),
        malasun_layer("hgrn2", 2, 72, 24, 88), malasun_layer("attention", 4, 40, 32, 0, 2, 2, 75, kv_from=0),
        malasun_layer("attention", 6, 64, 64, 120, 6, 1, 33, 0.17)]),
}


def malasun_config(raw: dict) -> dict:
    """A Malasun config.json -> the configuration the library takes."""
    layers = []
    for i, entry in enumerate(raw["layers"]):
        kind, mix, mlp = entry["type"], entry["mixer"], entry.get("mlp")
        if kind not in MIXER_IDS:
            raise _lib.RaiB200Error(-7, f"layer {i}: mixer {kind!r} is not implemented")
        if mlp is not None and mlp.get("kind", "dense") != "dense":
            raise _lib.RaiB200Error(-7, f"layer {i}: feed-forward kind {mlp['kind']!r} is not implemented")
        ff = int(mlp["ff"]) if mlp is not None else 0
        if kind == "attention":
            src = mix.get("kv_from")
            layers.append(malasun_layer(kind, int(mix["heads"]), int(mix["dim"]), int(mix["vdim"]), ff, int(mix["kv_heads"]),
                                        int(mix["conv"]), int(mix["mask"]["size"]), float(mix["scale"]),
                                        None if src is None else int(src)))
        else:
            layers.append(malasun_layer(kind, int(mix["heads"]), int(mix["dim"]), int(mix["vdim"]), ff))
    return _malasun(int(raw["vocab"]), int(raw["width"]), layers, float(raw["norm"]["eps"]))


def votapel_layer(heads: int, kv_heads: int, dim: int, ff: int = 0, experts: int = 0, top: int = 0, groups: int = 1,
                  keep: int = 1, router_scale: float = 1.0, shared_ff: int = 0, scale: float = 0.0, softcap: float = 0.0,
                  temp_coef: float = 0.0, temp_every: int = 0) -> dict:
    """One entry of a Votapel configuration's `layers`: attention whose values are its keys beside routed experts of inner size
    ff (0 leaves the feed-forward out) and a shared one (shared_ff).  softcap = 0 and temp_every = 0 leave those out."""
    mixer = dict(type="attention", heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=scale or dim ** -0.5, softcap=softcap,
                 temp_coef=temp_coef, temp_every=temp_every)
    mlp = dict(kind="moe", ff=ff, experts=experts, top=top, groups=groups, keep=keep, router_scale=router_scale,
               shared_ff=shared_ff) if ff else None
    return dict(mixer=mixer, mlp=mlp)


def _votapel(vocab: int, width: int, layers, max_positions: int, eps: float = 1e-6, residual_mult: float = 1.0) -> dict:
    return dict(arch="votapel", vocab_size=vocab, hidden_size=width, norm_eps=eps, max_positions=max_positions,
                residual_mult=residual_mult, layers=layers)


VOTAPEL: Dict[str, dict] = {
    # sizes that resemble a real model's layers, for throughput measurements (random weights)
    "votapel-1k": _votapel(32000, 1024, [votapel_layer(8, 2, 128, 512, 64, 4, 8, 4, 2.0, 1024, softcap=30.0, temp_coef=0.1,
                                                       temp_every=1024)] * 16, 8192, residual_mult=0.7),
    "votapel-2k": _votapel(32000, 2048, [votapel_layer(16, 4, 128, 1024, 32, 4, 4, 2, 2.0, 2048, softcap=30.0, temp_coef=0.1,
                                                       temp_every=1024)] * 12, 8192, residual_mult=0.7),
    "votapel-4k": _votapel(32000, 4096, [votapel_layer(32, 8, 128, 2048, 16, 2, 4, 2, 2.0, 4096, softcap=30.0, temp_coef=0.1,
                                                       temp_every=1024)] * 6, 8192, residual_mult=0.7),
    # a small model for tests
    "tiny-votapel": _votapel(352, 144, [
        votapel_layer(4, 2, 40, 56, 8, 2, 4, 2, 1.7, 72, softcap=9.0, temp_coef=0.3, temp_every=19),
        votapel_layer(6, 2, 64, 96, 15, 4, 5, 3, 0.8, 0, 0.11, temp_coef=0.6, temp_every=7),
        votapel_layer(3, 3, 24, softcap=20.0)], 400, 1e-5, 0.6),
}


def votapel_config(raw: dict) -> dict:
    """A Votapel config.json -> the configuration the library takes."""
    layers = []
    for i, entry in enumerate(raw["layers"]):
        kind, mix, mlp = entry["type"], entry["mixer"], entry.get("mlp")
        if kind != "attention":
            raise _lib.RaiB200Error(-7, f"layer {i}: mixer {kind!r} is not implemented")
        if int(mix["vdim"]) != int(mix["dim"]):
            raise _lib.RaiB200Error(-7, f"layer {i}: the values are the keys, so vdim must be dim")
        ff = {}
        if mlp is not None:
            if mlp.get("kind", "moe") != "moe":
                raise _lib.RaiB200Error(-7, f"layer {i}: feed-forward kind {mlp['kind']!r} is not implemented")
            router, groups, shared = mlp["router"], mlp["router"].get("groups") or {}, mlp.get("shared") or {}
            ff = dict(ff=int(mlp["expert"]["ff"]), experts=int(router["experts"]), top=int(router["top"]),
                      groups=int(groups.get("count", 1)), keep=int(groups.get("keep", 1)),
                      router_scale=float(router.get("scale", 1.0)), shared_ff=int(shared.get("ff", 0)))
        temp = mix.get("q_temp") or {}
        layers.append(votapel_layer(int(mix["heads"]), int(mix["kv_heads"]), int(mix["dim"]), scale=float(mix["scale"]),
                                    softcap=float(mix.get("softcap") or 0.0), temp_coef=float(temp.get("coef", 0.0)),
                                    temp_every=int(temp.get("every", 0)), **ff))
    return _votapel(int(raw["vocab"]), int(raw["width"]), layers, int(raw["max_positions"]), float(raw["norm"]["eps"]),
                    float(raw.get("residual_mult", 1.0)))


def rotation(dims: int, base: float, factor: float = 1.0, low: float = 1.0, high: float = 4.0, original: int = 0) -> dict:
    """Rotary positions on the first `dims` dimensions of a head.  original > 0: pairs that turn fewer than `low` times over
    that many positions have their frequency divided by `factor`, those that turn more than `high` times keep it."""
    scaling = dict(factor=factor, low=low, high=high, original=original) if original else None
    return dict(dims=dims, base=base, scaling=scaling)


def kufulix_attention(heads: int, kv_heads: int, dim: int, vdim: int = 0, window: int = 0, chunk: int = 0, rot=None, scale: float = 0.0,
                      qk_norm: bool = False, head_gate: bool = True) -> dict:
    """Attention within a sliding window or within chunks of the sequence."""
    return dict(type="attention", heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim or dim, window=window, chunk=chunk, rot=rot,
                scale=scale or dim ** -0.5, qk_norm=qk_norm, head_gate=head_gate, left_scale=1.0, ssd=None)


def kufulix_parallel(attention: dict, heads: int, vdim: int, state: int, groups: int = 1, conv: int = 4, norm_groups: int = 1,
                     left_scale: float = 1.0, right_scale: float = 1.0) -> dict:
    """Attention beside a Mamba-2 recurrence, on the same input."""
    return dict(attention, type="attention_ssd", left_scale=left_scale,
                ssd=dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=norm_groups, scale=right_scale))


def kufulix_experts(ff: int, experts: int, top: int, groups: int = 1, keep: int = 1, identity: int = 0) -> dict:
    """Routed experts of inner size ff; the last `identity` of the router's outputs return their input."""
    return dict(kind="moe", ff=ff, experts=experts, top=top, groups=groups, keep=keep, identity=identity)


def kufulix_layer(mixer: dict, mlp=None, weights_of=None) -> dict:
    """One entry of a Kufulix configuration's `layers`; weights_of names the layer whose tensors it uses."""
    return dict(mixer=mixer, mlp=mlp, weights_of=weights_of)


def _kufulix(vocab: int, width: int, layers, eps: float = 1e-6, logit_softcap: float = 0.0) -> dict:
    return dict(arch="kufulix", vocab_size=vocab, hidden_size=width, norm_eps=eps, logit_softcap=logit_softcap, layers=layers)


def _kufulix_bench(vocab: int, width: int, heads: int, kv_heads: int, ff: int, experts: int, top: int, groups: int, keep: int,
                   identity: int, pairs: int) -> dict:
    """Alternating layers of windowed attention beside a recurrence of twice the width, and of chunked attention; every
    second pair uses the weights of the one before it."""
    left = kufulix_attention(heads, kv_heads, 128, window=1024, rot=rotation(128, 1e4, 8.0, original=8192), qk_norm=True, head_gate=False)
    mixers = [kufulix_parallel(left, width // 32, 64, 128, left_scale=0.7, right_scale=0.7),
              kufulix_attention(heads, kv_heads, 128, chunk=3072, rot=rotation(128, 5e5, 8.0, original=8192))]
    mlp = kufulix_experts(ff, experts, top, groups, keep, identity)
    return _kufulix(vocab, width, [kufulix_layer(mixers[i], mlp, 2 * p - 2 + i if p % 2 else None) for p in range(pairs) for i in (0, 1)],
                    logit_softcap=30.0)


KUFULIX: Dict[str, dict] = {
    # sizes that resemble a real model's layers, for throughput measurements (random weights)
    "kufulix-1k": _kufulix_bench(32000, 1024, 8, 2, 512, 60, 4, 8, 4, 4, 8),
    "kufulix-2k": _kufulix_bench(32000, 2048, 16, 4, 1024, 30, 4, 4, 2, 2, 6),
    "kufulix-4k": _kufulix_bench(32000, 4096, 32, 8, 2048, 14, 2, 4, 2, 2, 4),
    # a small model for tests
    "tiny-kufulix": _kufulix(336, 152, [
        kufulix_layer(kufulix_parallel(kufulix_attention(4, 2, 40, 24, window=27, rot=rotation(16, 1e3, 3.0, 1.0, 3.0, 96), scale=0.21,
                                                         qk_norm=True, head_gate=False), 4, 32, 40, 2, 4, 2, 0.8, 1.3),
                      kufulix_experts(48, 7, 3, 3, 2, 2)),
        kufulix_layer(kufulix_attention(6, 2, 32, 56, chunk=50, rot=rotation(32, 5e3, 5.0, 0.5, 6.0, 64)), kufulix_experts(40, 8, 2, 4, 2, 0)),
        kufulix_layer(kufulix_attention(3, 3, 24, chunk=33, rot=rotation(8, 1e4)))], 1e-5, 12.0),
}
KUFULIX["tiny-kufulix"]["layers"] += [dict(KUFULIX["tiny-kufulix"]["layers"][i], weights_of=i) for i in (0, 1)]


def _kufulix_attention_config(mix: dict, windowed: bool) -> dict:
    """The attention part of a mixer's entry: a sliding window and q/k norm, or chunks and a gate per head."""
    rot, size = mix.get("rot"), int(mix["mask"]["size"])
    if rot:
        s = rot.get("scaling")
        rot = rotation(int(rot["dims"]), float(rot["base"]), *((float(s["factor"]), float(s["low"]), float(s["high"]), int(s["original"])) if s else ()))
    return kufulix_attention(int(mix["heads"]), int(mix["kv_heads"]), int(mix["dim"]), int(mix["vdim"]), size if windowed else 0,
                             0 if windowed else size, rot, float(mix["scale"]), windowed, not windowed)


def kufulix_config(raw: dict) -> dict:
    """A Kufulix config.json -> the configuration the library takes."""
    layers = []
    for i, entry in enumerate(raw["layers"]):
        kind, mix, mlp = entry["type"], entry["mixer"], entry.get("mlp")
        if kind == "attention":
            mixer = _kufulix_attention_config(mix, False)
        elif kind == "parallel":
            r = mix["right"]
            mixer = kufulix_parallel(_kufulix_attention_config(mix["left"], True), int(r["heads"]), int(r["vdim"]), int(r["state"]),
                                     int(r["groups"]), int(r["conv"]), int(r["norm_groups"]), float(mix["left_scale"]),
                                     float(mix["right_scale"]))
        else:
            raise _lib.RaiB200Error(-7, f"layer {i}: mixer {kind!r} is not implemented")
        if mlp is not None:
            if mlp.get("kind", "moe") != "moe":
                raise _lib.RaiB200Error(-7, f"layer {i}: feed-forward kind {mlp['kind']!r} is not implemented")
            router, groups = mlp["router"], mlp["router"].get("groups") or {}
            mlp = kufulix_experts(int(mlp["expert"]["ff"]), int(router["experts"]), int(router["top"]), int(groups.get("count", 1)),
                                  int(groups.get("keep", 1)), int(router.get("identity") or 0))
        src = entry.get("weights_of")
        layers.append(kufulix_layer(mixer, mlp, None if src is None else int(src)))
    return _kufulix(int(raw["vocab"]), int(raw["width"]), layers, float(raw["norm"]["eps"]), float(raw.get("logit_softcap") or 0.0))


def yarn_rotation(dims: int, base: float, factor: float = 0.0, fast: float = 32.0, slow: float = 1.0, original: int = 0,
                  interleaved: bool = False) -> dict:
    """Rotary positions on the first `dims` dimensions, neighbours paired (interleaved) or halves.  original > 0: pairs that turn
    fewer than about `slow` times over that many positions have their frequency divided by `factor`, those that turn more than
    about `fast` times keep it, and the turned vectors grow by 0.1 ln(factor) + 1 (YaRN)."""
    scaling = dict(factor=factor, fast=fast, slow=slow, original=original) if original else None
    return dict(dims=dims, base=base, scaling=scaling, interleaved=interleaved)


def fizadra_attention(heads: int, kv_heads: int, dim: int, vdim: int = 0, rot=None, scale: float = 0.0) -> dict:
    """Causal attention whose heads' scores are mixed before a softmax with one added to its denominator."""
    return dict(type="attention", heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim or dim, rot=rot, scale=scale or dim ** -0.5)


def fizadra_latent(heads: int, dim: int, rot_dim: int, vdim: int, q_rank: int, kv_rank: int, rot=None, scale: float = 0.0,
                   sink: bool = False, gate: str = "heads", kv_from=None) -> dict:
    """Causal attention over a cached latent; gate: one number per output element ("elements") or per head ("heads"); kv_from
    names the earlier layer whose latent it reads."""
    return dict(type="latent_attention", heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank,
                rot=rot or yarn_rotation(rot_dim, 1e4), scale=scale or (dim + rot_dim) ** -0.5, sink=sink, gate=gate, kv_from=kv_from)


def fizadra_layer(mixer: dict, ff: int = 0) -> dict:
    """One entry of a Fizadra configuration's `layers`; ff = 0 leaves the feed-forward out."""
    return dict(mixer=mixer, mlp=dict(kind="dense", ff=ff) if ff else None)


def _fizadra(vocab: int, width: int, layers, groups: int = 1, eps: float = 1e-6) -> dict:
    return dict(arch="fizadra", vocab_size=vocab, hidden_size=width, norm_eps=eps, norm_groups=groups, layers=layers)


def _fizadra_bench(vocab: int, width: int, heads: int, kv_heads: int, kv_rank: int, ff: int, quads: int) -> dict:
    """Layers in fours: latent attention with sinks, attention with mixed heads, and two of latent attention with a gate per head;
    the sinks' layer of every second four reads the latent of the one before it."""
    layers = []
    for n in range(quads):
        rot = yarn_rotation(32, 1e4, 8.0, original=4096, interleaved=True)
        layers.append(fizadra_latent(heads, 96, 32, 128, width // 2, kv_rank, rot, sink=True, gate="elements",
                                     kv_from=4 * n - 4 if n % 2 else None))
        layers.append(fizadra_attention(heads, kv_heads, 128, rot=yarn_rotation(128, 5e5)))
        layers += [fizadra_latent(heads, 96, 32, 128, width // 2, kv_rank, yarn_rotation(32, 5e5))] * 2
    return _fizadra(vocab, width, [fizadra_layer(m, ff) for m in layers], 4)


FIZADRA: Dict[str, dict] = {
    # sizes that resemble a real model's layers, for throughput measurements (random weights)
    "fizadra-1k": _fizadra_bench(32000, 1024, 8, 2, 256, 4096, 4),
    "fizadra-2k": _fizadra_bench(32000, 2048, 16, 4, 512, 8192, 3),
    "fizadra-4k": _fizadra_bench(32000, 4096, 32, 8, 512, 16384, 2),
    # a small model for tests
    "tiny-fizadra": _fizadra(328, 168, [
        fizadra_layer(fizadra_latent(3, 24, 16, 40, 56, 72, yarn_rotation(16, 700.0, 5.0, 9.0, 0.5, 90, True), 0.19, True, "elements"), 104),
        fizadra_layer(fizadra_attention(6, 2, 40, 56, yarn_rotation(24, 2e3), 0.21), 96),
        fizadra_layer(fizadra_latent(5, 32, 8, 24, 48, 40, yarn_rotation(8, 3e3)), 72),
        fizadra_layer(fizadra_latent(4, 16, 16, 32, 40, 72, yarn_rotation(16, 700.0, 5.0, 9.0, 0.5, 90, True), 0.25, True, "elements", 0)),
        fizadra_layer(fizadra_attention(4, 4, 24, 24, yarn_rotation(24, 1e4)), 88)], 3, 1e-5),
}


def _fizadra_rotation(rot, interleaved: bool):
    if not rot:
        return None
    s = rot.get("scaling")
    return yarn_rotation(int(rot["dims"]), float(rot["base"]), *((float(s["factor"]), float(s["fast"]), float(s["slow"]),
                                                                  int(s["original"])) if s else ()), interleaved=interleaved)


def fizadra_config(raw: dict) -> dict:
    """A Fizadra config.json -> the configuration the library takes."""
    layers = []
    for i, entry in enumerate(raw["layers"]):
        kind, mix, mlp = entry["type"], entry["mixer"], entry.get("mlp")
        if kind == "attention":
            mixer = fizadra_attention(int(mix["heads"]), int(mix["kv_heads"]), int(mix["dim"]), int(mix["vdim"]),
                                      _fizadra_rotation(mix.get("rot"), False), float(mix["scale"]))
        elif kind in ("latent_attention", "latent_attention_2"):
            first, src = kind == "latent_attention", mix.get("kv_from")   # the first kind: neighbours turn, sinks, a gate per element
            mixer = fizadra_latent(int(mix["heads"]), int(mix["dim"]), int(mix["rot_dim"]), int(mix["vdim"]), int(mix["q_rank"]),
                                   int(mix["kv_rank"]), _fizadra_rotation(mix["rot"], first), float(mix["scale"]), first,
                                   "elements" if first else "heads", None if src is None else int(src))
        else:
            raise _lib.RaiB200Error(-7, f"layer {i}: mixer {kind!r} is not implemented")
        if mlp is not None and mlp.get("kind", "dense") != "dense":
            raise _lib.RaiB200Error(-7, f"layer {i}: feed-forward kind {mlp['kind']!r} is not implemented")
        layers.append(fizadra_layer(mixer, int(mlp["ff"]) if mlp is not None else 0))
    norm = raw["norm"]
    return _fizadra(int(raw["vocab"]), int(raw["width"]), layers, int(norm.get("groups") or 1), float(norm["eps"]))


# by config.json's `architecture`
_CONFIG_READERS = {"Malasun": malasun_config, "Votapel": votapel_config, "Kufulix": kufulix_config, "Fizadra": fizadra_config}
_MODEL_TYPES = {"qwen2": "qwen2", "phi": "phi2", "phi2": "phi2", "phi3": "phi3", "gemma": "gemma"}


def from_json(path: str) -> dict:
    """The configuration in a checkpoint folder's (or file's) config.json, whichever architecture it names."""
    if os.path.isdir(path):
        path = os.path.join(path, "config.json")
    with open(path) as f:
        raw = json.load(f)
    reader = _CONFIG_READERS.get(raw.get("architecture"))
    if reader:
        return reader(raw)
    name = raw.get("arch") or _MODEL_TYPES.get(raw.get("model_type"))
    if name not in ARCH_IDS or name in LAYERED:
        raise _lib.RaiB200Error(-7, f"{path}: architecture {raw.get('architecture') or raw.get('model_type')!r} is not implemented")
    return dict(raw, arch=name)


def get(name: str) -> dict:
    src = BASELINE.get(name) or TINY.get(name) or MALASUN.get(name) or VOTAPEL.get(name) or KUFULIX.get(name) or FIZADRA.get(name)
    if src is None:
        raise KeyError(f"unknown configuration {name!r}")
    return copy.deepcopy(src)


def head_dim(cfg: dict) -> int:
    return cfg["hidden_size"] // cfg["num_attention_heads"]


def rotary_dim(cfg: dict) -> int:
    # phi2.rs:47: (partial_rotary_factor * head_dim) as usize
    return int(cfg.get("partial_rotary_factor", 1.0) * head_dim(cfg))


def norm_eps(cfg: dict) -> float:
    return cfg["layer_norm_eps"] if cfg["arch"] == "phi2" else cfg["rms_norm_eps"]


def tied(cfg: dict) -> bool:
    return cfg["arch"] == "gemma" or bool(cfg.get("tie_word_embeddings", False))


def layer_structs(cfg: dict):
    """The rb_layer_config array of a layer-by-layer configuration."""
    arr = (_lib.LayerConfig * len(cfg["layers"]))()
    for s, layer in zip(arr, cfg["layers"]):
        mix, mlp = layer["mixer"], layer["mlp"]
        s.mixer = MIXER_IDS[mix["type"]]
        s.heads, s.key_dim, s.value_dim = mix["heads"], mix["dim"], mix["vdim"]
        s.kv_from = s.weights_of = -1
        s.mlp_size = mlp["ff"] if mlp else 0
        if cfg["arch"] == "fizadra":
            s.block, s.scale, s.mlp_kind = _lib.BLOCK_SANDWICH, mix["scale"], _lib.MLP_DENSE_RELU2
            r = mix["rot"]
            if r:
                s.rot_dims, s.rot_base, s.rot_interleaved = r["dims"], r["base"], int(r["interleaved"])
                if r["scaling"]:
                    r = r["scaling"]
                    s.rot_yarn, s.rot_original, s.rot_factor, s.rot_low, s.rot_high = 1, r["original"], r["factor"], r["slow"], r["fast"]
            if mix["type"] == "attention":
                s.kv_heads, s.qk_norm, s.talk, s.softmax_one = mix["kv_heads"], 1, 1, 1
            else:
                s.kv_heads, s.rot_dim, s.q_rank, s.kv_rank = 1, mix["rot_dim"], mix["q_rank"], mix["kv_rank"]
                s.sink, s.head_gate = int(mix["sink"]), int(mix["gate"] == "heads")
                s.kv_from = -1 if mix["kv_from"] is None else mix["kv_from"]
        elif cfg["arch"] == "kufulix":
            s.block = _lib.BLOCK_PRE_NORM
            s.weights_of = -1 if layer.get("weights_of") is None else layer["weights_of"]
            s.kv_heads, s.scale, s.window, s.chunk = mix["kv_heads"], mix["scale"], mix["window"], mix["chunk"]
            s.qk_norm, s.head_gate, s.mixer_scale = int(mix["qk_norm"]), int(mix["head_gate"]), mix["left_scale"]
            if mix["rot"]:
                s.rot_dims, s.rot_base = mix["rot"]["dims"], mix["rot"]["base"]
                if mix["rot"]["scaling"]:
                    r = mix["rot"]["scaling"]
                    s.rot_original, s.rot_factor, s.rot_low, s.rot_high = r["original"], r["factor"], r["low"], r["high"]
            if mix["ssd"]:
                r = mix["ssd"]
                s.ssd_heads, s.ssd_value_dim, s.ssd_state, s.ssd_groups = r["heads"], r["vdim"], r["state"], r["groups"]
                s.ssd_norm_groups, s.conv_taps, s.ssd_scale = r["norm_groups"], r["conv"], r["scale"]
            if mlp:
                s.mlp_kind, s.experts, s.top, s.identity = _lib.MLP_EXPERTS_RELU2, mlp["experts"], mlp["top"], mlp["identity"]
                s.groups, s.keep_groups = mlp["groups"], mlp["keep"]
        elif cfg["arch"] == "votapel":
            s.block, s.residual_mult = _lib.BLOCK_PARALLEL, cfg["residual_mult"]
            s.kv_heads, s.scale, s.softcap = mix["kv_heads"], mix["scale"], mix["softcap"]
            s.temp_coef, s.temp_every = mix["temp_coef"], mix["temp_every"]
            if mlp:
                s.mlp_kind, s.experts, s.top = _lib.MLP_EXPERTS, mlp["experts"], mlp["top"]
                s.groups, s.keep_groups = mlp["groups"], mlp["keep"]
                s.router_scale, s.shared_size = mlp["router_scale"], mlp["shared_ff"]
        elif mix["type"] == "attention":
            s.kv_heads, s.conv_taps, s.window, s.scale = mix["kv_heads"], mix["conv"], mix["window"], mix["scale"]
            s.kv_from = -1 if mix["kv_from"] is None else mix["kv_from"]
    return arr


def create_model(ctx, cfg: dict, struct, out) -> None:
    """rb_model_create or rb_model_create_layers, by architecture."""
    if cfg["arch"] in LAYERED:
        _lib.call("rb_model_create_layers", ctx, ctypes.byref(struct), ctypes.byref(layer_structs(cfg)), ctypes.byref(out))
    else:
        _lib.call("rb_model_create", ctx, ctypes.byref(struct), ctypes.byref(out))


def to_struct(cfg: dict, dtype: int, max_batch: int, max_seq: int, max_tokens: int, tp_rank: int = 0,
              tp_size: int = 1) -> "_lib.ModelConfig":
    if cfg["arch"] == "phi2" and cfg.get("qk_layernorm"):
        raise _lib.RaiB200Error(-7, "phi2 qk_layernorm is not implemented (phi2.rs:166-172)")
    s = _lib.ModelConfig()
    s.arch = ARCH_IDS[cfg["arch"]]
    s.dtype = dtype
    s.max_batch, s.max_seq, s.max_tokens = int(max_batch), int(max_seq), int(max_tokens)
    s.tp_rank, s.tp_size = int(tp_rank), int(tp_size)
    if cfg["arch"] in LAYERED:
        s.vocab_size, s.hidden_size, s.num_hidden_layers = cfg["vocab_size"], cfg["hidden_size"], len(cfg["layers"])
        s.max_position_embeddings = cfg.get("max_positions", 0)
        s.norm_eps, s.logit_softcap, s.norm_groups = cfg["norm_eps"], cfg.get("logit_softcap", 0.0), cfg.get("norm_groups", 1)
        return s
    for k in ("vocab_size", "hidden_size", "intermediate_size", "num_hidden_layers", "num_attention_heads",
              "max_position_embeddings"):
        setattr(s, k, int(cfg[k]))
    s.num_key_value_heads = int(cfg.get("num_key_value_heads") or cfg["num_attention_heads"])
    s.rotary_dim = rotary_dim(cfg)
    s.hidden_act = ACT_IDS[cfg["hidden_act"]]
    s.tie_word_embeddings = int(tied(cfg))
    # only qwen2's mask has the sliding-window term (qwen2.rs:316-327); the other families' masks are plain causal
    s.sliding_window = int(cfg.get("sliding_window") or 0) if cfg["arch"] == "qwen2" else 0
    s.rope_theta = float(cfg["rope_theta"])
    s.norm_eps = float(norm_eps(cfg))
    return s
