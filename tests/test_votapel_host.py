"""Votapel without a GPU: the configuration reader, the parameter list, and the plain oracle against independent forms."""
import json
import math

import numpy as np
import pytest
import votapel_ref as ref
from votapel_util import decided_weights, raw_config

from rai_b200 import _lib, configs, synth
from rai_b200.configs import votapel_layer as layer


def small():
    return dict(arch="votapel", vocab_size=90, hidden_size=56, norm_eps=1e-3, max_positions=50, residual_mult=0.8, layers=[
        layer(6, 3, 16, 40, 12, 3, 4, 2, 1.3, 24, 0.3, 7.0, 0.4, 5), layer(2, 1, 24, scale=0.2),
        layer(4, 4, 8, 16, 5, 5, router_scale=0.5)])


def test_config_json_is_read_whole(tmp_path):
    cfg = small()
    (tmp_path / "config.json").write_text(json.dumps(raw_config(cfg)))
    assert configs.from_json(str(tmp_path)) == cfg
    s = configs.layer_structs(cfg)
    assert all(x.block == _lib.BLOCK_PARALLEL and x.residual_mult == 0.8 and x.kv_from == -1 for x in s)
    assert [x.mlp_size for x in s] == [40, 0, 16] and [x.shared_size for x in s] == [24, 0, 0]
    assert (s[0].heads, s[0].kv_heads, s[0].key_dim, s[0].value_dim, s[0].scale, s[0].softcap) == (6, 3, 16, 16, 0.3, 7.0)
    assert (s[0].temp_coef, s[0].temp_every, s[0].experts, s[0].top, s[0].groups, s[0].keep_groups) == (0.4, 5, 12, 3, 4, 2)
    assert (s[0].mlp_kind, s[0].router_scale, s[2].router_scale) == (_lib.MLP_EXPERTS, 1.3, 0.5)
    assert (s[1].softcap, s[1].temp_every, s[2].groups, s[2].keep_groups) == (0.0, 0, 1, 1)
    st = configs.to_struct(cfg, _lib.F32, 3, 100, 200)
    assert (st.arch, st.num_hidden_layers, st.max_position_embeddings, st.vocab_size, st.hidden_size) == (_lib.ARCH_VOTAPEL, 3, 50, 90, 56)
    assert abs(st.norm_eps - 1e-3) < 1e-12


@pytest.mark.parametrize("change", [lambda e: e.update(type="mamba"), lambda e: e["mlp"].update(kind="dense"),
                                    lambda e: e["mixer"].update(vdim=8)])
def test_what_is_not_implemented_is_refused(change):
    raw = raw_config(small())
    change(raw["layers"][0])
    with pytest.raises(_lib.RaiB200Error):
        configs.votapel_config(raw)


def test_attention_options_struct_matches_header():
    import re
    body = re.search(r"typedef struct rb_attention_options \{(.*?)\} rb_attention_options;", _lib.HEADER.read_text(), flags=re.S).group(1)
    body = re.sub(r"/\*.*?\*/", "", body, flags=re.S)
    fields = [ln.split()[-1].strip("*;") for ln in body.splitlines() if ln.strip().endswith(";")]
    assert fields == [f[0] for f in _lib.AttentionOptions._fields_]


def test_parameter_list():
    cfg = small()
    shapes = {n: s for n, s, _ in synth.param_shapes(cfg)}
    assert shapes["pos"] == (50, 56) and shapes["l0.norm1"] == (56,) and shapes["final.norm"] == (56,)
    assert shapes["l0.mix.q"] == (96, 56) and shapes["l0.mix.k.b"] == (48,) and shapes["l0.mix.sink"] == (6,) and shapes["l0.mix.o"] == (56, 96)
    assert shapes["l0.mlp.e11.down"] == (56, 40) and shapes["l0.mlp.router"] == (12, 56) and shapes["l0.mlp.shared.up"] == (24, 56)
    assert not any(n.startswith("l1.mlp") for n in shapes) and "l2.mlp.shared.up" not in shapes and "l0.mix.v" not in shapes
    w = synth.weights(cfg, 1)
    assert all(np.asarray(w[n]).shape == s for n, s in shapes.items())


def test_query_temperature_steps_at_whole_stretches():
    t = [ref.query_temperature(p, 0.5, 4) for p in range(12)]
    assert t[:3] == [1.0] * 3 and t[3] == t[6] == 1 + 0.5 * math.log(2) and t[7] == 1 + 0.5 * math.log(3) and t[11] == 1 + 0.5 * math.log(4)


def test_sink_takes_weight_and_gives_no_value():
    s = np.array([0.3, -1.0, 2.0])
    p = ref.sink_softmax(s, 1.5)
    np.testing.assert_allclose(p, np.exp(s) / (np.exp(s).sum() + math.exp(1.5)), rtol=1e-12)
    np.testing.assert_allclose(ref.sink_softmax(s, -1e9).sum(), 1.0)
    assert ref.sink_softmax(s, 700.0).sum() < 1e-200


def test_attention_against_a_dense_form():
    rng = np.random.default_rng(2)
    T, H, G = 19, 6, 2
    q, k = rng.standard_normal((T, H, 8)) * 3, rng.standard_normal((T, G, 8))
    sink = rng.standard_normal(H)
    got = ref.attention(q, k, k, 0.4, 5.0, sink)
    for h in range(H):
        s = 5.0 * np.tanh(q[:, h] @ k[:, h // 3].T * 0.4 / 5.0)
        e = np.where(np.tril(np.ones((T, T))) > 0, np.exp(s), 0.0)
        np.testing.assert_allclose(got[:, h], e / (e.sum(1, keepdims=True) + np.exp(sink[h])) @ k[:, h // 3], atol=1e-12)
    np.testing.assert_allclose(ref.attention(q[12:], k, k, 0.4, 5.0, sink, first=12), got[12:], atol=1e-12)


def test_experts_are_chosen_within_the_strongest_groups():
    s = np.array([.9, .1, .1, .8, .7, .1, .6, .65, .66])       # strengths 1.0, 1.5, 1.31
    assert ref.chosen_experts(s, 2, 3, 1) == [3, 4]             # the single best expert is in a group that is out
    assert ref.chosen_experts(s, 4, 3, 2) == [3, 4, 8, 7]
    assert ref.chosen_experts(s, 3, 1, 1) == [0, 3, 4]
    assert ref.chosen_experts(s, 2, 9, 2) == [0, 3]             # groups of one


def test_parallel_block_prefixes_and_decided_weights():
    """A position does not depend on what follows; the test weights' choices keep a margin in the model itself."""
    cfg = small()
    w = ref.as_float64(decided_weights(cfg, 3))
    toks = np.random.default_rng(4).integers(0, 90, 40)
    full = ref.logits(cfg, w, toks)
    np.testing.assert_allclose(ref.logits(cfg, w, toks[:17]), full[:17], atol=1e-10)
    x = ref.embed(w, toks)
    for i, stream in enumerate(ref.residual_streams(cfg, w, toks)):
        mlp = cfg["layers"][i]["mlp"]
        if mlp:
            s = ref.sigmoid(ref.rms_norm_one_plus(x, w[f"l{i}.norm1"], cfg["norm_eps"]) @ w[f"l{i}.mlp.router"].T)
            noisy = ref.sigmoid(ref.rms_norm_one_plus(x, w[f"l{i}.norm1"], cfg["norm_eps"]) * 1.004 @ w[f"l{i}.mlp.router"].T)
            picks = [ref.chosen_experts(a, mlp["top"], mlp["groups"], mlp["keep"]) for a in s]
            assert picks == [ref.chosen_experts(a, mlp["top"], mlp["groups"], mlp["keep"]) for a in noisy]
            assert len({e for p in picks for e in p}) == mlp["experts"]
        x = stream


def test_benchmark_compares_models_of_equal_size():
    import os
    import sys
    sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    import bench
    for name in ("votapel-1k", "votapel-2k", "votapel-4k"):
        cfg = configs.get(name)
        other, ours, theirs = bench.equal_size_qwen2(cfg)
        assert abs(ours - theirs) < 0.03 * ours
        assert other["num_hidden_layers"] == len(cfg["layers"]) and other["hidden_size"] == cfg["hidden_size"]
        assert configs.head_dim(other) == 128
        lean, active, theirs = bench.equal_size_qwen2(cfg, active=True)
        assert abs(active - theirs) < 0.03 * active and active < 0.5 * ours and lean["intermediate_size"] < other["intermediate_size"]
