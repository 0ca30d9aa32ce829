"""Fizadra without a GPU: the configuration reader, the parameter list, and the plain oracle against independent forms."""
import json
import math
import re

import fizadra_ref as ref
import numpy as np
import pytest
from fizadra_util import pointed, raw_config

from rai_b200 import _lib, configs, synth
from rai_b200.configs import fizadra_attention, fizadra_latent, fizadra_layer, yarn_rotation


def small(groups=2):
    yarn = yarn_rotation(10, 80.0, 4.0, 3.0, 0.5, 50, True)
    return configs._fizadra(61, 36, [
        fizadra_layer(fizadra_latent(3, 14, 10, 18, 22, 20, yarn, 0.3, True, "elements"), 44),
        fizadra_layer(fizadra_attention(6, 2, 16, 12, yarn_rotation(10, 300.0), 0.2)),
        fizadra_layer(fizadra_latent(2, 8, 10, 6, 12, 20, yarn, 0.4, True, "elements", 0), 30),
        fizadra_layer(fizadra_latent(5, 6, 4, 10, 16, 8, yarn_rotation(4, 40.0), 0.25), 28)], groups, 1e-4)


def test_config_json_is_read_whole(tmp_path):
    cfg = small()
    raw = raw_config(cfg)
    (tmp_path / "config.json").write_text(json.dumps(raw))
    assert configs.from_json(str(tmp_path)) == cfg
    assert [e["type"] for e in raw["layers"]] == ["latent_attention", "attention", "latent_attention", "latent_attention_2"]
    s = configs.layer_structs(cfg)
    assert all(x.block == _lib.BLOCK_SANDWICH and x.mlp_kind == _lib.MLP_DENSE_RELU2 and x.weights_of == -1 for x in s)
    assert [x.mixer for x in s] == [_lib.MIXER_LATENT, _lib.MIXER_ATTENTION, _lib.MIXER_LATENT, _lib.MIXER_LATENT]
    assert [x.kv_from for x in s] == [-1, -1, 0, -1] and [x.mlp_size for x in s] == [44, 0, 30, 28]
    assert (s[0].heads, s[0].key_dim, s[0].rot_dim, s[0].value_dim, s[0].q_rank, s[0].kv_rank, s[0].scale) == (3, 14, 10, 18, 22, 20, 0.3)
    assert [(x.sink, x.head_gate) for x in s] == [(1, 0), (0, 0), (1, 0), (0, 1)]
    assert (s[0].rot_interleaved, s[0].rot_yarn, s[0].rot_dims, s[0].rot_base, s[0].rot_factor, s[0].rot_low, s[0].rot_high, s[0].rot_original) == (
        1, 1, 10, 80.0, 4.0, 0.5, 3.0, 50)
    assert (s[3].rot_interleaved, s[3].rot_yarn, s[3].rot_dims, s[3].rot_base) == (0, 0, 4, 40.0)
    assert (s[1].heads, s[1].kv_heads, s[1].key_dim, s[1].value_dim, s[1].talk, s[1].softmax_one, s[1].qk_norm) == (6, 2, 16, 12, 1, 1, 1)
    st = configs.to_struct(cfg, _lib.F32, 3, 100, 200)
    assert (st.arch, st.num_hidden_layers, st.vocab_size, st.hidden_size, st.norm_groups) == (_lib.ARCH_FIZADRA, 4, 61, 36, 2)
    raw["norm"].pop("groups")
    assert configs.fizadra_config(raw)["norm_groups"] == 1


@pytest.mark.parametrize("change", [lambda e: e.update(type="mamba"), lambda e: e["mlp"].update(kind="experts")])
def test_what_is_not_implemented_is_refused(change):
    raw = raw_config(small())
    change(raw["layers"][0])
    with pytest.raises(_lib.RaiB200Error):
        configs.fizadra_config(raw)


@pytest.mark.parametrize("name,struct", [("rb_layer_config", "LayerConfig"), ("rb_model_config", "ModelConfig"),
                                         ("rb_attention_options", "AttentionOptions")])
def test_structs_match_header(name, struct):
    body = re.search(r"typedef struct %s \{(.*?)\} %s;" % (name, name), _lib.HEADER.read_text(), flags=re.S).group(1)
    body = re.sub(r"/\*.*?\*/|//[^\n]*", "", body, flags=re.S)
    fields = []
    for decl in body.split(";"):
        for part in decl.split(","):
            if part.strip():
                fields.append(re.split(r"[\s*]+", part.strip())[-1])
    assert fields == [f[0] for f in getattr(_lib, struct)._fields_]


def test_parameter_list():
    cfg = small()
    shapes = {n: s for n, s, _ in synth.param_shapes(cfg)}
    assert shapes["l0.mix.dq"] == (22, 36) and shapes["l0.mix.uq"] == (72, 22) and shapes["l0.mix.dkv"] == (30, 36)
    assert shapes["l0.mix.dkv.norm"] == (20,) and shapes["l0.mix.uk"] == (42, 20) and shapes["l0.mix.uv"] == (54, 20)
    assert shapes["l0.mix.sink"] == (3,) and shapes["l0.mix.g"] == (54, 36) and shapes["l3.mix.g"] == (5, 36) and "l3.mix.sink" not in shapes
    assert "l2.mix.dkv" not in shapes and shapes["l2.mix.uk"] == (16, 20)
    assert shapes["l1.mix.q"] == (96, 36) and shapes["l1.mix.v.b"] == (24,) and shapes["l1.mix.talk"] == (6, 6) and shapes["l1.mix.o"] == (36, 72)
    assert not any(n.startswith(("l1.mlp", "l1.norm2")) for n in shapes) and shapes["l1.norm1b"] == shapes["l0.norm2b"] == (36,)
    assert [shapes[f"l{i}.dwa"] for i in range(4)] == [(2,), (3,), (4,), (5,)] and shapes["head"] == (61, 36)
    w = synth.weights(cfg, 1)
    assert all(np.asarray(w[n]).shape == s for n, s in shapes.items())


def test_frequencies_have_three_ranges():
    rot = yarn_rotation(32, 1e3, 8.0, 6.0, 0.8, 256)
    plain, f = ref.rotary_frequencies(yarn_rotation(32, 1e3)), ref.rotary_frequencies(rot)
    at = [32 * math.log(256 / (2 * math.pi * n)) / (2 * math.log(1e3)) for n in (6.0, 0.8)]   # where a pair turns so often
    lo, hi = math.floor(at[0]), math.ceil(at[1])
    assert 0 < lo < hi < 16
    assert f[:lo + 1] == plain[:lo + 1] and all(abs(f[i] - plain[i] / 8) < 1e-15 for i in range(hi, 16))
    assert all(plain[i] / 8 < f[i] < plain[i] for i in range(lo + 1, hi)) and all(a > b for a, b in zip(f, f[1:]))
    assert abs(ref.rotary_amplitude(rot) - (1 + 0.1 * math.log(8))) < 1e-15 and ref.rotary_amplitude(yarn_rotation(32, 1e3)) == 1.0


@pytest.mark.parametrize("interleaved", [False, True])
def test_rotation_against_complex_numbers(interleaved):
    rng = np.random.default_rng(0)
    rot = yarn_rotation(12, 100.0, 3.0, 2.0, 0.3, 30, interleaved)
    q, k = rng.standard_normal((1, 1, 20)), rng.standard_normal((1, 1, 20))
    dot = lambda i, j: float((ref.rotate(q, rot, i) * ref.rotate(k, rot, j)).sum())  # noqa: E731
    assert abs(dot(7, 3) - dot(107, 103)) < 1e-9 and abs(dot(7, 3) - dot(7, 4)) > 1e-3
    r = ref.rotate(q, rot, 5)
    np.testing.assert_array_equal(r[..., 12:], q[..., 12:])
    first, second = (slice(0, 12, 2), slice(1, 12, 2)) if interleaved else (slice(0, 6), slice(6, 12))
    turn = ref.rotary_amplitude(rot) * np.exp(5j * np.array(ref.rotary_frequencies(rot)))
    z = (q[0, 0, first] + 1j * q[0, 0, second]) * turn
    np.testing.assert_allclose(r[0, 0, first] + 1j * r[0, 0, second], z, atol=1e-12)


@pytest.mark.parametrize("with_sink,with_talk", [(False, False), (True, False), (True, True)])
def test_attention_against_a_dense_form(with_sink, with_talk):
    rng = np.random.default_rng(2)
    T, H, G = 19, 6, 2
    q, k, v = rng.standard_normal((T, H, 8)) * 3, rng.standard_normal((T, G, 8)), rng.standard_normal((T, G, 5))
    sink = rng.standard_normal(H) if with_sink else None
    talk = rng.standard_normal((H, H)) if with_talk else None
    got = ref.attention(q, k, v, 0.4, sink, talk)
    s = np.einsum("thd,nhd->htn", q, np.repeat(k, 3, 1)) * 0.4
    s = np.einsum("hg,gtn->htn", talk, s) if with_talk else s
    e = np.exp(s) * np.tril(np.ones((T, T)))
    total = e.sum(-1, keepdims=True) + (np.exp(sink)[:, None, None] if with_sink else 0.0)
    np.testing.assert_allclose(got, np.einsum("htn,nhe->the", e / total, np.repeat(v, 3, 1)), atol=1e-12)
    np.testing.assert_allclose(ref.attention(q[12:], k, v, 0.4, sink, talk, first=12), got[12:], atol=1e-12)


def test_softmax_with_one_added_is_a_sink_of_zero():
    s = np.array([-40.0, -41.0, -39.5])
    p = ref.softmax_with_sink(s, 0.0)
    np.testing.assert_allclose(p, np.exp(s) / (1 + np.exp(s).sum()))
    assert p.sum() < 1e-15 and abs(ref.softmax_with_sink(s).sum() - 1) < 1e-15


def test_latent_attention_in_the_latents_space():
    """Queries moved into the latents' space and results moved out of it: what a single token computes."""
    cfg = small()
    mix, w = cfg["layers"][0]["mixer"], ref.as_float64(synth.weights(cfg, 3))
    rng = np.random.default_rng(3)
    h, p, T, H = rng.standard_normal((17, 36)), "l0.mix", 17, 3
    c, turned = ref.latent(h, w, p, mix, 1e-4)
    want = ref.latent_attention_mixer(h, w, p, mix, 1e-4, c, turned)
    u = h @ w[p + ".dq"].T
    u = u / np.sqrt((u * u).mean(1, keepdims=True) + 1e-4) * w[p + ".dq.norm"]
    q = (u @ w[p + ".uq"].T).reshape(T, H, 24)
    rows = np.einsum("thd,hdr->thr", q[..., :14], w[p + ".uk"].reshape(H, 14, 20))
    rows = np.concatenate([rows, ref.rotate(q[..., 14:], mix["rot"])], -1)
    e = np.einsum("thr,nr->htn", rows, np.concatenate([c, turned], 1)) * 0.3
    e = np.exp(e) * np.tril(np.ones((T, T)))
    o = np.einsum("htn,nr->thr", e / (e.sum(-1, keepdims=True) + np.exp(w[p + ".sink"])[:, None, None]), c)
    o = np.einsum("thr,her->the", o, w[p + ".uv"].reshape(H, 18, 20)).reshape(T, -1) / (1 + np.exp(-(h @ w[p + ".g"].T)))
    np.testing.assert_allclose(o @ w[p + ".o"].T, want, atol=1e-10)


def test_group_norm_and_depth_average():
    rng = np.random.default_rng(4)
    x, w = rng.standard_normal((3, 12)), rng.standard_normal(12)
    got = ref.group_norm(x, w, 3, 0.0) / w
    np.testing.assert_allclose((got.reshape(3, 3, 4) ** 2).mean(-1), 1.0)
    np.testing.assert_allclose(ref.group_norm(x, w, 1, 0.01), x / np.sqrt((x * x).mean(-1, keepdims=True) + 0.01) * w)
    xs = rng.standard_normal((4, 3, 12))
    c = rng.standard_normal(4)
    np.testing.assert_allclose(ref.depth_average(c, list(xs)), np.einsum("i,itw->tw", c, xs), atol=1e-12)


def test_history_holds_results_before_they_are_averaged():
    cfg = small()
    w = ref.as_float64(synth.weights(cfg, 5))
    for i in range(4):      # every layer hands on the embedding alone: nothing a layer adds is seen
        w[f"l{i}.dwa"] = np.eye(i + 2)[0] * 2.0
    toks = [3, 9, 1]
    assert all(np.allclose(x, 2.0 * w["embed"][toks]) for x in ref.residual_streams(cfg, w, toks))


def test_prefixes_and_pointed_weights():
    """A position does not depend on what follows; the pointed weights make one far key matter in the whole model."""
    cfg = small()
    w = ref.as_float64(pointed(cfg, synth.weights(cfg, 6), 7, 11))
    toks = np.random.default_rng(6).integers(12, 61, 40)
    toks[0], toks[39] = 11, 7
    full = ref.logits(cfg, w, toks)
    np.testing.assert_allclose(ref.logits(cfg, w, toks[:17]), full[:17], atol=1e-10)
    toks[0] = 13
    other = ref.logits(cfg, w, toks)
    assert np.sqrt(np.mean((other[39] - full[39]) ** 2)) > 0.1 * np.sqrt(np.mean(full[39] ** 2))


def test_benchmark_compares_models_of_equal_size():
    import os
    import sys
    sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    import bench
    for name in ("fizadra-1k", "fizadra-2k", "fizadra-4k"):
        cfg = configs.get(name)
        assert {x["mixer"]["type"] for x in cfg["layers"]} == {"attention", "latent_attention"}
        other, ours, theirs = bench.equal_size_qwen2(cfg)
        assert abs(ours - theirs) < 0.03 * ours and ours == bench.param_count(cfg)
        assert other["num_hidden_layers"] == len(cfg["layers"]) and other["hidden_size"] == cfg["hidden_size"]
        assert bench.relatives(name, cfg)["malasun"]["hidden_size"] == cfg["hidden_size"]
