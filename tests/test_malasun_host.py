"""Malasun without a GPU: the configuration reader, the parameter list, and the plain oracle against independent forms."""
import json

import malasun_ref as ref
import numpy as np
import pytest

from rai_b200 import _lib, configs, synth

RAW = {
    "architecture": "Malasun", "vocab": 96, "width": 48, "norm": {"eps": 1e-5},
    "layers": [
        {"type": "attention", "mixer": {"heads": 6, "kv_heads": 3, "dim": 16, "vdim": 24, "conv": 5, "scale": 0.3,
                                        "mask": {"size": 9}}, "mlp": None},
        {"type": "hgrn2", "mixer": {"heads": 2, "dim": 24, "vdim": 40}, "mlp": {"kind": "dense", "ff": 72}},
        {"type": "attention", "mixer": {"heads": 6, "kv_heads": 3, "dim": 16, "vdim": 24, "conv": 2, "scale": 0.2,
                                        "mask": {"size": 31}, "kv_from": 0}, "mlp": {"kind": "dense", "ff": 56}},
    ],
}


def test_config_json_is_read_whole(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(RAW))
    cfg = configs.from_json(str(tmp_path))
    assert (cfg["arch"], cfg["vocab_size"], cfg["hidden_size"], cfg["norm_eps"]) == ("malasun", 96, 48, 1e-5)
    s = configs.layer_structs(cfg)
    assert [x.mixer for x in s] == [_lib.MIXER_ATTENTION, _lib.MIXER_HGRN2, _lib.MIXER_ATTENTION]
    assert [x.kv_from for x in s] == [-1, -1, 0]
    assert [x.mlp_size for x in s] == [0, 72, 56]
    assert (s[0].heads, s[0].kv_heads, s[0].key_dim, s[0].value_dim, s[0].conv_taps, s[0].window, s[0].scale) == (6, 3, 16, 24, 5, 9, 0.3)
    assert (s[1].heads, s[1].key_dim, s[1].value_dim) == (2, 24, 40)
    assert (s[2].conv_taps, s[2].window, s[2].scale) == (2, 31, 0.2)
    st = configs.to_struct(cfg, _lib.F32, 3, 100, 200)
    assert (st.arch, st.dtype, st.num_hidden_layers, st.max_batch, st.max_seq, st.max_tokens) == (_lib.ARCH_MALASUN, _lib.F32, 3, 3, 100, 200)
    assert abs(st.norm_eps - 1e-5) < 1e-12


def test_what_is_not_implemented_is_refused(tmp_path):
    bad = json.loads(json.dumps(RAW))
    bad["layers"][0]["type"] = "mamba"
    with pytest.raises(_lib.RaiB200Error):
        configs.malasun_config(bad)
    bad = json.loads(json.dumps(RAW))
    bad["layers"][1]["mlp"]["kind"] = "experts"
    with pytest.raises(_lib.RaiB200Error):
        configs.malasun_config(bad)
    (tmp_path / "config.json").write_text(json.dumps({"model_type": "unheard-of"}))
    with pytest.raises(_lib.RaiB200Error):
        configs.from_json(str(tmp_path))


def test_other_architectures_are_read_by_model_type(tmp_path):
    hf = dict(configs.get("tiny-qwen2"))
    hf.pop("arch")
    (tmp_path / "config.json").write_text(json.dumps(dict(hf, model_type="qwen2")))
    assert configs.from_json(str(tmp_path))["arch"] == "qwen2"


def test_parameter_list():
    shapes = {n: s for n, s, _ in synth.param_shapes(configs.malasun_config(RAW))}
    assert shapes["l0.mix.q"] == (96, 48) and shapes["l0.mix.v"] == (72, 48) and shapes["l0.mix.k.conv"] == (48, 5)
    assert shapes["l0.mix.k.norm"] == (48,) and "l0.mix.v.norm" not in shapes and "l0.norm2" not in shapes
    assert shapes["l1.mix.lower"] == (48,) and shapes["l1.mix.norm"] == (40,) and shapes["l1.mlp.act"] == (2,)
    assert "l2.mix.k" not in shapes and "l2.mix.v.conv" not in shapes and shapes["l2.mix.q.conv"] == (96, 2)
    assert shapes["final.norm"] == () and shapes["head"] == (96, 48)
    w = synth.weights(configs.malasun_config(RAW), 1)
    assert all(np.asarray(w[n]).shape == s for n, s in shapes.items())


def test_safetensors_round_trip_keeps_single_numbers(tmp_path):
    from rai_b200 import safetensors_io
    w = synth.weights(configs.malasun_config(RAW), 2)
    path = str(tmp_path / "m.safetensors")
    safetensors_io.write_safetensors(path, w, "BF16")
    with safetensors_io.SafetensorsFile(path) as f:
        got = {n: s for n, _, s, _ in f.entries}
    assert got["l0.norm1"] == () and got["l0.mix.q.conv"] == (96, 5)


def test_convolution_against_numpy():
    rng = np.random.default_rng(0)
    u, taps = rng.standard_normal((11, 3)), rng.standard_normal((3, 4))
    for c in range(3):
        want = np.convolve(u[:, c], taps[c, ::-1])[:11]
        np.testing.assert_allclose(ref.causal_conv(u, taps)[:, c], want, atol=1e-12)


def test_recurrence_against_its_unrolled_sum():
    rng = np.random.default_rng(1)
    q, v = rng.standard_normal((9, 5)), rng.standard_normal((9, 4))
    f = rng.uniform(0.2, 0.99, (9, 5))
    o, _ = ref.gated_linear_recurrence(q, f, v)
    for t in range(9):
        want = sum(((q[t] * (1 - f[s]) * np.prod(f[s + 1:t + 1], axis=0)).sum()) * v[s] for s in range(t + 1))
        np.testing.assert_allclose(o[t], want, atol=1e-12)


def test_attention_against_a_dense_mask():
    rng = np.random.default_rng(2)
    T, H, G, window = 23, 6, 2, 7
    q, k, v = rng.standard_normal((T, H, 8)), rng.standard_normal((T, G, 8)), rng.standard_normal((T, G, 5))
    got = ref.window_attention(q, k, v, 0.4, ref.alibi_slopes(H), window)
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    for h in range(H):
        s = q[:, h] @ k[:, h // 3].T * 0.4 - 2.0 ** (-8 * (h + 1) / H) * (i - j)
        s = np.where((j <= i) & (j > i - window), s, -np.inf)
        p = np.exp(s - s.max(1, keepdims=True))
        np.testing.assert_allclose(got[:, h], p / p.sum(1, keepdims=True) @ v[:, h // 3], atol=1e-12)


def test_activation_is_smooth_and_odd_sizes_work():
    pq = np.array([0.4, -0.7])
    z = np.array([-30.0, -1.0, -1e-4, 0.0, 1e-4, 2.0])
    y = ref.xielu(z, pq)
    assert abs(y[3]) == 0 and abs(y[2] + 0.5e-4) < 1e-7 and abs(y[4] - 0.5e-4) < 1e-7
    np.testing.assert_allclose(y[5], np.log1p(np.exp(0.4)) * 4 + 1.0, rtol=1e-12)
    np.testing.assert_allclose(y[0], (0.5 + np.log1p(np.exp(-0.7))) * (np.exp(-30.0) - 1 + 30.0) - 15.0, rtol=1e-12)


def test_shared_keys_and_prefixes():
    """A position's logits do not depend on what follows it, and a layer with kv_from reads that layer's keys."""
    cfg = configs.malasun_config(RAW)
    w = ref.as_float64(synth.weights(cfg, 3))
    toks = np.random.default_rng(4).integers(0, 96, 40)
    full = ref.logits(cfg, w, toks)
    np.testing.assert_allclose(ref.logits(cfg, w, toks[:17]), full[:17], atol=1e-10)
    changed = dict(w, **{"l0.mix.k": w["l0.mix.k"] * 1.5})
    a, b = ref.residual_streams(cfg, w, toks), ref.residual_streams(cfg, changed, toks)
    assert np.abs(a[2] - b[2]).max() > np.abs(a[1] - b[1]).max() * 0.1 > 0


def test_benchmark_compares_models_of_equal_size():
    import os
    import sys
    sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    import bench
    for name in ("malasun-1k", "malasun-2k", "malasun-4k"):
        cfg = configs.get(name)
        other, ours, theirs = bench.equal_size_qwen2(cfg)
        assert abs(ours - theirs) < 0.02 * ours
        assert other["num_hidden_layers"] == len(cfg["layers"]) and other["hidden_size"] == cfg["hidden_size"]
        assert configs.head_dim(other) == 128
