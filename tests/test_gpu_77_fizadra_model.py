"""The Fizadra design through the framework's own model, scheduler and entry points, against the plain oracle."""
import json
import os
import subprocess
import sys

import fizadra_ref as ref
import numpy as np
import pytest
import torch
from fizadra_util import pointed, raw_config
from malasun_util import DTYPES, rms_err

from rai_b200 import _lib, configs, safetensors_io, synth
from rai_b200.configs import fizadra_attention as attention
from rai_b200.configs import fizadra_latent as latent
from rai_b200.configs import fizadra_layer as layer
from rai_b200.configs import yarn_rotation
from rai_b200.models import Model

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {_lib.BF16: 4e-2, _lib.F32: 3e-5}


def cfg_of(name):
    if name == "tiny":
        return configs.get("tiny-fizadra")
    if name == "odd":          # nothing is a multiple of 8; layers without a feed-forward; latents used twice, by both kinds
        yarn, plain = yarn_rotation(6, 90.0, 3.0, 4.0, 0.5, 40, True), yarn_rotation(10, 60.0)
        return configs._fizadra(203, 75, [
            layer(latent(5, 13, 6, 20, 33, 45, yarn, 0.3, True, "elements"), 61), layer(attention(6, 3, 20, 31, yarn_rotation(14, 90.0), 0.25)),
            layer(latent(3, 21, 10, 9, 18, 30, plain, 0.2), 50), layer(latent(7, 9, 6, 11, 27, 45, yarn, 0.4, True, "elements", 0)),
            layer(latent(2, 15, 10, 13, 50, 30, plain, 0.22, kv_from=2), 35), layer(attention(3, 1, 37, 12, None, 0.17), 44)], 5, 1e-3)
    if name == "wide-heads":   # the tcgen05 prefill kernel (keys of 64 and of 128), a large latent, many mixed heads
        return configs._fizadra(256, 256, [
            layer(latent(4, 96, 32, 128, 128, 512, yarn_rotation(32, 1e4, 8.0, 32.0, 1.0, 256, True), 0.09, True, "elements"), 512),
            layer(attention(16, 4, 128, 64, yarn_rotation(64, 1e5)), 320), layer(latent(8, 32, 32, 64, 96, 128, yarn_rotation(32, 1e4)), 256),
            layer(attention(8, 8, 64, 128, yarn_rotation(64, 1e4)), 256)], 4, 1e-6)
    if name == "plain":        # every constant that can be neutral is
        return configs._fizadra(128, 64, [layer(latent(1, 32, 32, 32, 32, 32), 64), layer(attention(1, 1, 32, 32, yarn_rotation(32, 1e4)), 64)], 1)
    if name == "large-heads":  # heads that only the mma.sync and the latents' kernels take; more mixed heads than the joint kernel
        return configs._fizadra(128, 96, [layer(latent(2, 144, 56, 72, 40, 200, yarn_rotation(56, 1e3, 2.0, 8.0, 1.0, 64, True), 0.1, True, "elements"), 64),
                                          layer(attention(36, 36, 16, 16, yarn_rotation(8, 1e3))), layer(latent(2, 250, 64, 40, 24, 72, yarn_rotation(64, 1e3)), 64),
                                          layer(latent(70, 16, 8, 16, 48, 64, yarn_rotation(8, 1e3)))], 3, 1e-5)
    raise KeyError(name)


NAMES = ["tiny", "odd", "wide-heads", "plain", "large-heads"]
_made = {}


def weights_of(name):
    if name not in _made:
        w = synth.weights(cfg_of(name), 7)
        _made[name] = (w, ref.as_float64(w))
    return _made[name]


def build(name, dtype, cuda, batch=4, max_seq=400, max_tokens=1600):
    m = Model(cfg_of(name), dtype, cuda, batch, max_seq, max_tokens)
    m.update_params(weights_of(name)[0])
    return m.cfg, m, weights_of(name)[1]


def tokens(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab_size"], n)


def close(got, want, dtype):
    """Every position: root mean square over the vocabulary relative to that of the logits at large."""
    got, want = got.double().cpu().numpy(), np.asarray(want)
    err = np.sqrt(((got - want) ** 2).mean(-1)) / np.sqrt((want ** 2).mean())
    assert err.max() < TOL[dtype] and np.median(err) < 0.5 * TOL[dtype], (err.argmax(), err.max(), np.median(err))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompt(cuda, name, dtype):
    cfg, m, w = build(name, dtype, cuda)
    t = tokens(cfg, 200, 1)
    close(m.forward_rows(t[None], None, range(200), 0), ref.logits(cfg, w, t), dtype)
    m.clear_kv_cache()
    assert m.logits_dtype == torch.float32
    one = m.forward(t[None, :3], 0)    # Model::fwd: the last position only
    close(one[:, 0], ref.logits(cfg, w, t[:3])[-1:], dtype)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["tiny", "odd", "wide-heads"])
def test_residual_stream_after_every_layer(cuda, name, dtype):
    cfg, m, w = build(name, dtype, cuda)
    t = tokens(cfg, 60, 2)
    got = m.forward_layers(t[None])
    for i, want in enumerate(ref.residual_streams(cfg, w, t)):
        assert rms_err(got[i], want) < (1.5e-2 if dtype == _lib.BF16 else 3e-6), i
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_portions_and_single_tokens(cuda, name, dtype):
    """The same tokens in portions of many sizes, down to two tokens and one: multiplied-out latents against the latents' space."""
    cfg, m, w = build(name, dtype, cuda)
    t = tokens(cfg, 150, 3)
    want = ref.logits(cfg, w, t)
    for sizes in ([64, 64, 22], [2] * 75, [100, 1, 1, 1, 2, 45], [1] * 150, [3, 120, 27]):
        m.clear_kv_cache()
        at, got = 0, []
        for n in sizes:
            got.append(m.forward_rows(t[None, at:at + n], None, range(n)))
            at += n
        close(torch.cat(got), want, dtype)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["tiny", "odd", "wide-heads"])
def test_unequal_requests_join_leave_and_reuse_slots(cuda, name, dtype):
    """Requests of different lengths in one batch, some ending, new ones joining on the pages given back."""
    cfg, m, w = build(name, dtype, cuda, batch=3)
    text = {k: tokens(cfg, 150, 10 + i) for i, k in enumerate("abcde")}
    want = {k: ref.logits(cfg, w, t) for k, t in text.items()}
    live, held = [], {}

    def step(feed):
        """feed: request -> how many tokens.  New requests go behind the live ones."""
        live.extend(k for k in feed if k not in live)
        n = max(max(feed.values()), 1)
        ids, lens, rows, who = np.zeros((len(live), n), dtype=np.int64), [], [], []
        for b, k in enumerate(live):
            c, at = feed.get(k, 0), held.get(k, 0)
            ids[b, :c] = text[k][at:at + c]
            ids[b, c:] = 5 + b                       # padding must not show
            lens.append(c)
            rows += [b * n + s for s in range(c)]
            who += [(k, at + s) for s in range(c)]
            held[k] = at + c
        close(m.forward_rows(ids, lens, rows), np.stack([want[k][p] for k, p in who]), dtype)

    def end(*gone):
        m.keep_sequences([b for b, k in enumerate(live) if k not in gone])
        for k in gone:
            live.remove(k)

    step({"a": 70, "b": 1, "c": 33})
    for _ in range(4):
        step({"a": 1, "b": 1, "c": 1})
    end("b")
    step({"a": 1, "c": 1})
    step({"a": 1, "c": 1, "d": 40})                  # a prompt beside single tokens
    step({"a": 1, "d": 2})                           # c waits
    step({"a": 65, "c": 1, "d": 1})
    end("a", "d")
    step({"c": 1, "e": 1})                           # a request of one token on used pages
    for _ in range(30):
        step({"c": 1, "e": 1})
    end("c", "e")
    live.clear()
    held.clear()
    step({"e": 129})
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_large_decode_batch(cuda, dtype):
    """Three hundred sequences of single tokens: more rows than the split-K form takes."""
    cfg, m, w = build("wide-heads", dtype, cuda, batch=300, max_seq=64, max_tokens=1200)
    text = np.stack([tokens(cfg, 5, 100 + b) for b in range(300)])
    m.forward_rows(text[:, :3], None, [], 0)
    for at in (3, 4):
        got = m.forward_rows(text[:, at:at + 1], None, range(0, 300, 23))
    close(got, np.stack([ref.logits(cfg, w, text[b])[4] for b in range(0, 300, 23)]), dtype)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["tiny", "wide-heads"])
def test_rows_do_not_depend_on_the_batch(cuda, name, dtype):
    """Alone, or beside other requests: the same logits up to rounding."""
    cfg, m, _ = build(name, dtype, cuda)
    a, b, c = (tokens(cfg, n, 20 + i) for i, n in enumerate((50, 120, 90)))
    alone = m.forward_rows(a[None], None, [49], 0)
    m.clear_kv_cache()
    ids = np.full((3, 120), 3)
    ids[0, :120], ids[1, :50], ids[2, :90] = b, a, c
    both = m.forward_rows(ids, [120, 50, 90], [120 + 49], 0)
    close(both, alone.double().cpu().numpy(), dtype)
    m.close()


def pointing():
    """Every kind of layer, the turning part short of the dimension that points."""
    yarn = yarn_rotation(8, 1e3, 4.0, 8.0, 0.5, 64, True)
    cfg = configs._fizadra(96, 104, [layer(latent(2, 24, 8, 24, 32, 40, yarn, 0.2, True, "elements"), 48),
                                     layer(attention(4, 2, 32, 24, yarn_rotation(16, 1e4), 0.2)),
                                     layer(latent(2, 16, 16, 32, 24, 32, yarn_rotation(16, 1e3), 0.2), 40),
                                     layer(latent(2, 24, 8, 24, 32, 40, yarn, 0.2, True, "elements", 0))], 2, 1e-5)
    return cfg, pointed(cfg, synth.weights(cfg, 9), 94, 95)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cut", ["prompt", "decoded", "portion"])
def test_a_far_key(cuda, dtype, cut):
    """One key token looked for by one query token: far away, at page borders, in the first position, right before it."""
    cfg, w = pointing()
    w64 = ref.as_float64(w)
    m = Model(cfg, dtype, cuda, 1, 400, 400)
    m.update_params(w)
    base = np.random.default_rng(1).integers(0, 94, 290)
    for row, key in ((129, 0), (128, 127), (128, 64), (250, 1), (279, 63), (280, 64), (191, 190), (192, 64), (64, 63), (65, 64), (1, 0), (33, 31)):
        t = base[:row + 1].copy()
        t[key] = 95
        t[row] = 94
        want = ref.logits(cfg, w64, t)[-1:]
        m.clear_kv_cache()
        n = row + 1
        if cut == "prompt":
            got = m.forward_rows(t[None], None, [row], 0)
        else:
            lead = n - 1 if cut == "decoded" else max(1, n - 7)
            m.forward_rows(t[None, :lead], None, [], 0)
            got = m.forward_rows(t[None, lead:], None, [n - lead - 1])
        close(got, want, dtype)
        plain = t.copy()                             # (the oracle: that key shows)
        plain[key] = base[key]
        assert np.abs(ref.logits(cfg, w64, plain)[-1] - want[0]).max() > 0.3 * np.sqrt((want ** 2).mean()), (row, key)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("what", ["sink", "talk", "dwa", "norm1b", "g", "dkv.norm", "amplitude"])
def test_each_weight_shows(cuda, dtype, what):
    """A change of one kind of weight changes the model as it changes the oracle, and by enough to be seen."""
    cfg, w = cfg_of("tiny"), dict(weights_of("tiny")[0])
    t = tokens(cfg, 90, 4)
    before = ref.logits(cfg, weights_of("tiny")[1], t)
    if what == "amplitude":
        cfg = json.loads(json.dumps(cfg))
        for i in (0, 3):
            cfg["layers"][i]["mixer"]["rot"]["scaling"]["factor"] = 60.0
    else:
        rng = np.random.default_rng(5)
        for n in w:
            if n.endswith("." + what) or n.endswith(".mix." + what):
                w[n] = synth.bf16_round(np.asarray(w[n] + (4.0 if what == "sink" else rng.standard_normal(w[n].shape) * 0.5), dtype=np.float32)).reshape(w[n].shape)
    want = ref.logits(cfg, ref.as_float64(w), t)
    moved = np.sqrt(((want - before) ** 2).mean(-1)) / np.sqrt((want ** 2).mean())
    assert moved.max() > 2 * TOL[dtype]
    m = Model(cfg, dtype, cuda, 1, 128, 128)
    m.update_params(w)
    lead = m.forward_rows(t[None, :70], None, range(70), 0)
    close(torch.cat([lead] + [m.forward_rows(t[None, i:i + 1], None, [0]) for i in range(70, 90)]), want, dtype)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["tiny", "wide-heads"])
def test_long_greedy_generation(cuda, name, dtype):
    """The captured decode loop over many pages: its tokens against plain steps and against the oracle."""
    cfg, m, w = build(name, dtype, cuda, batch=2, max_seq=420)
    prompt = np.stack([tokens(cfg, 30, 31), tokens(cfg, 30, 32)])
    out = m.generate(prompt, 230)
    assert _lib.lib().rb_model_decode_graph_active(m._m) == 1
    plain, logits = m.greedy_generate(prompt, 40, collect_logits=True)
    assert (out[:, :40] == plain.numpy()).all()
    for b in range(2):
        text = np.concatenate([prompt[b], out[b]])
        want = ref.logits(cfg, w, text[:-1])[29:]
        # a token may differ from the oracle's choice only where the oracle's own margin is within the tolerance
        chosen = want[np.arange(len(want)), out[b]]
        assert (want.max(1) - chosen < 4 * TOL[dtype] * np.sqrt((want ** 2).mean())).all()
        close(logits[:, b], want[:40], dtype)
        assert len(set(out[b].tolist())) > 5
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_ragged_generation_and_sampling(cuda, dtype):
    cfg, m, w = build("tiny", dtype, cuda)
    prompts = [tokens(cfg, n, 40 + n) for n in (3, 77, 41)]
    out = m.generate_ragged(prompts, 50)
    for b, p in enumerate(prompts):
        want = ref.logits(cfg, w, np.concatenate([p, out[b]])[:-1])[len(p) - 1:]
        chosen = want[np.arange(50), out[b]]
        assert (want.max(1) - chosen < 4 * TOL[dtype] * np.sqrt((want ** 2).mean())).all()
    m.set_sampling(1e9, 64, -1)
    pen = m.generate_ragged(prompts, 30)
    for row in pen:
        assert len(set(row.tolist())) == 30     # nothing within the window repeats
    m.set_sampling(0.0, 0, int(out[1][4]))
    stop = m.generate_ragged(prompts, 30)
    first = out[1].tolist().index(out[1][4])
    assert (stop[1][first:] == out[1][4]).all() and m.finished(3)[1]
    m.close()


@pytest.fixture(scope="module")
def checkpoint(tmp_path_factory):
    folder = tmp_path_factory.mktemp("fizadra")
    cfg = json.loads(json.dumps(cfg_of("odd")))
    cfg["layers"][5]["mixer"]["rot"] = yarn_rotation(36, 1e3)    # (the file always names a rotation)
    w = synth.weights(cfg, 7)
    (folder / "config.json").write_text(json.dumps(raw_config(cfg)))
    safetensors_io.write_safetensors(str(folder / "model.safetensors"), w, "BF16")
    return str(folder), cfg, ref.as_float64(w)


@pytest.mark.parametrize("dtype", DTYPES)
def test_checkpoint_folder(cuda, checkpoint, dtype, tmp_path):
    folder, cfg, w = checkpoint
    assert configs.from_json(folder) == cfg
    m = Model.from_pretrained(folder, dtype, cuda, 1, 64)
    t = tokens(cfg, 40, 50)
    close(m.forward_rows(t[None], None, range(40), 0), ref.logits(cfg, w, t), dtype)
    path = str(tmp_path / "back.safetensors")
    m.to_safetensors(path)
    with safetensors_io.SafetensorsFile(path) as f, safetensors_io.SafetensorsFile(os.path.join(folder, "model.safetensors")) as g:
        shapes = {n: s for n, _, s, _ in g.entries}
        assert {n: s for n, _, s, _ in f.entries} == shapes
        if dtype == _lib.BF16:
            assert all(f.read_bytes(n) == g.read_bytes(n) for n in shapes)
    m.close()


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_runner(cuda, checkpoint, dtype, tmp_path):
    """bin/trace_run as a program: unequal prompts, single tokens, requests that end, a later and larger batch."""
    folder, cfg, w = checkpoint
    text = {k: tokens(cfg, n, 60 + i).tolist() for i, (k, n) in enumerate((("x", 40), ("y", 1), ("z", 70), ("u", 90), ("v", 9)))}
    want = {k: ref.logits(cfg, w, t) for k, t in text.items()}
    plan = [([("x", 35), ("y", 1), ("z", 66)], ["y"])] + [([("z", 1), ("x", 1)], [])] * 3 + [([("x", 1), ("z", 1)], ["x", "z"])]
    plan += [([("u", 88), ("v", 8)], []), ([("u", 1), ("v", 1)], ["v"]), ([("u", 1)], ["u"])]
    at, lines, expect = {}, [], {}
    for n, (feed, end) in enumerate(plan):
        entries, rows = [], []
        for k, c in feed:
            lo = at.get(k, 0)
            picks = [] if n == 1 else list(range(c - 1, -1, -2))      # a step that wants nothing, and unordered wants
            entries.append({"id": k, "tokens": text[k][lo:lo + c], "want": picks})
            rows += [want[k][lo + s] for s in picks]
            at[k] = lo + c
        lines.append(json.dumps({"step": n, "entries": entries, "end": end}))
        expect[n] = rows
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(tmp_path),
                        "--max-tokens", "128"], input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=120)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {n}" for n in range(len(plan))]
    for n, rows in expect.items():
        if rows:
            got = np.fromfile(tmp_path / f"{n}.f32", dtype="<f4").reshape(len(rows), cfg["vocab_size"])
            close(torch.from_numpy(got), np.stack(rows), _lib.BF16 if dtype == "bfloat16" else _lib.F32)


def test_command_line(cuda, checkpoint):
    folder, cfg, _ = checkpoint
    r = subprocess.run([sys.executable, "-m", "rai_b200", "generate", "--model", folder, "--dtype", "float32", "--prompt", "5,9,100",
                        "--prompt", "7", "--steps", "6"], cwd=ROOT, capture_output=True, text=True, timeout=120)
    assert r.returncode == 0, r.stderr
    m = Model.from_pretrained(folder, _lib.F32, cuda, 2, 64)
    want = m.generate_ragged([np.array([5, 9, 100]), np.array([7])], 6)
    m.close()
    assert [[int(t) for t in line.split(",")] for line in r.stdout.split()] == want.tolist()


def test_bad_shapes_are_refused(cuda):
    cfg = cfg_of("tiny")
    for at, path, value in ((1, ("mixer", "kv_heads"), 4), (1, ("mixer", "dim"), 300), (1, ("mixer", "rot", "dims"), 15), (1, ("mixer", "rot", "dims"), 48),
                            (1, ("mixer", "scale"), -1.0), (0, ("mixer", "rot", "dims"), 18), (0, ("mixer", "kv_rank"), 2000), (0, ("mixer", "q_rank"), -1),
                            (3, ("mixer", "kv_from"), 2), (3, ("mixer", "kv_from"), 3), (3, ("mixer", "kv_from"), 1), (3, ("mixer", "rot", "base"), 701.0),
                            (3, ("mixer", "kv_rank"), 80), (0, ("mlp", "ff"), -8)):
        bad = json.loads(json.dumps(cfg))
        part = bad["layers"][at]
        for k in path[:-1]:
            part = part[k]
        part[path[-1]] = value
        with pytest.raises(_lib.RaiB200Error):
            Model(bad, _lib.BF16, cuda, 1, 16)
    for key, value in (("norm_groups", 5), ("norm_groups", 0)):
        with pytest.raises(_lib.RaiB200Error):
            Model(dict(json.loads(json.dumps(cfg)), **{key: value}), _lib.BF16, cuda, 1, 16)
    with pytest.raises(_lib.RaiB200Error):
        Model(cfg, _lib.BF16, cuda, 1, 16, tp_rank=0, tp_size=2)
