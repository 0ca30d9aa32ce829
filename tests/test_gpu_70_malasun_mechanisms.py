"""Each mechanism of the Malasun design alone, through its C entry point, against the plain oracle."""
import ctypes

import malasun_ref as ref
import numpy as np
import pytest
import torch
from malasun_util import DTYPES, Cache, dev, pad8, padded, ptr, rms_err, rounded

from rai_b200 import _lib

pytestmark = pytest.mark.gpu
TOL = {_lib.BF16: 6e-3, _lib.F32: 2e-6}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,n,k", [(1, 24, 40), (9, 200, 72), (40, 136, 512), (150, 264, 64), (300, 136, 128)])
def test_xielu_epilogue(cuda, dtype, m, n, k):
    rng = np.random.default_rng(m)
    x, w = rounded(rng.standard_normal((m, k)), dtype), rounded(rng.standard_normal((n, k)) * 2 / np.sqrt(k), dtype)
    pq = rounded([0.7, -1.3], dtype)
    out = torch.empty((m, n), dtype=dev([0], dtype).dtype, device="cuda")
    xd, wd, pd = dev(x, dtype), dev(w, dtype), dev(pq, dtype)
    _lib.call("rb_linear_act", cuda.ctx, ptr(xd), ptr(wd), None, ptr(out), m, n, k, _lib.ACT_XIELU, ptr(pd), dtype)
    cuda.synchronize()
    assert rms_err(out, ref.xielu(x @ w.T, pq)) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,rows", [(52, 3), (320, 40), (2048, 700)])
def test_residual_stream(cuda, dtype, width, rows):
    """Embedding, the norm on a sublayer's output (from a tensor and from split-K slabs), the final norm."""
    rng, ld = np.random.default_rng(width), pad8(width)
    table = rounded(rng.standard_normal((77, width)), dtype)
    ids = rng.integers(0, 77, rows)
    h = torch.empty((rows, ld), device="cuda")
    x = torch.empty((rows, ld), dtype=dev([0], dtype).dtype, device="cuda")
    td, idd = dev(padded(table, ld), dtype), torch.from_numpy(ids.astype(np.int32)).cuda()
    _lib.call("rb_embed_stream", cuda.ctx, ptr(td), dtype, 77, width, ld, ptr(idd), rows, ptr(h), ptr(x))
    cuda.synchronize()
    assert (h.cpu().double().numpy()[:, :width] == table[ids]).all() and (x.float() == h).all()

    y, slabs = rounded(rng.standard_normal((rows, width)) * 3, dtype), rng.standard_normal((3, rows, width))
    gain = rounded([1.37], dtype)
    gd, yd, sd = dev(gain, dtype), dev(padded(y, ld), dtype), dev(np.stack([padded(s, ld) for s in slabs]), torch.float32)
    want = table[ids]
    for tensor, acc, sub in ((yd, None, y), (None, sd, slabs.sum(0))):
        _lib.call("rb_add_scaled_norm", cuda.ctx, ptr(tensor), ptr(acc), 0 if acc is None else 3, ptr(gd), 0.25, rows, width, ld,
                  ptr(h), ptr(x), dtype)
        want = want + ref.scalar_rms_norm(sub, gain, 0.25)
    cuda.synchronize()
    assert rms_err(h[:, :width], want) < 1e-6      # the stream is float32 in both dtypes
    assert rms_err(x[:, :width], want) < TOL[dtype] and (h[:, width:] == 0).all()

    pick = rng.integers(0, rows, 5)
    out = torch.empty((5, ld), dtype=x.dtype, device="cuda")
    rd = torch.from_numpy(pick.astype(np.int32)).cuda()
    _lib.call("rb_scalar_norm_rows", cuda.ctx, ptr(h), ptr(rd), 0, ptr(gd), 0.25, 5, width, ld, ptr(out), dtype)
    cuda.synchronize()
    assert rms_err(out[:, :width], ref.scalar_rms_norm(want[pick], gain, 0.25)) < TOL[dtype]


def conv_op(cuda, cache, dtype, src, conv, norms, heads, dims, batch, s_new, ring, q_pad, new_lens=None, bias=None, acc=None,
            taps=1, eps=1e-6, gate_out=None):
    (H, G), (d, e) = heads, dims
    q = torch.empty((batch * s_new, H, q_pad), dtype=dev([0], dtype).dtype, device="cuda")
    t = src if src is not None else acc
    _lib.call("rb_conv_norm_append", cuda.ctx, ptr(src), ptr(acc), 0 if acc is None else acc.shape[0], ptr(bias), ptr(conv), taps,
              ptr(norms[0]), ptr(norms[1]), eps, batch, s_new, H, G, d, e, t.shape[-1], cache.h, 0, ptr(ring), ptr(new_lens),
              ptr(q), ptr(gate_out), dtype)
    return q


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,e,taps", [(4, 2, 40, 32, 4), (3, 1, 20, 36, 2), (2, 2, 64, 64, 1), (5, 5, 12, 8, 7)])
def test_convolution_norm_and_append(cuda, dtype, H, G, d, e, taps):
    """A prompt, a portion of two tokens (its second row is padding for one sequence), then single tokens out of slabs."""
    rng = np.random.default_rng(H * d)
    B, eps, D = 2, 1e-3, pad8(max(d, e)) if dtype == _lib.F32 else 64
    nq, nk, nv, ng = H * d, G * d, G * e, H * e
    offs = np.cumsum([0, pad8(nq), pad8(nk), pad8(nv), pad8(ng)])
    cols = [np.arange(n) + o for n, o in zip((nq, nk, nv, ng), offs)]
    C, N = int(offs[3]), int(offs[4])
    lens = [9, 11]                     # tokens of each sequence in total
    steps = [(6, None), (2, [1, 2]), (1, None), (1, [1, 1]), (1, [0, 1])]
    u = [rounded(rng.standard_normal((lens[b], N)), dtype) for b in range(B)]
    w = {n: rounded(rng.standard_normal((c, taps)), dtype) for n, c in (("q", nq), ("k", nk), ("v", nv))}
    norm = {n: rounded(1 + 0.3 * rng.standard_normal(c), dtype) for n, c in (("q", nq), ("k", nk))}
    want = []
    for b in range(B):
        y = {n: ref.causal_conv(u[b][:, c], w[n]) for n, c in zip("qkv", cols)}
        for n in "qk":
            y[n] = ref.rms_normalise(y[n], eps) * norm[n]
        want.append(y)
    conv = np.zeros((taps, C))
    for n, c in zip("qkv", cols):
        conv[:, c] = w[n].T
    convd = dev(conv, dtype)
    nd = [dev(np.pad(norm["q"], (0, pad8(nq) - nq)), dtype), dev(np.pad(norm["k"], (0, pad8(nk) - nk)), dtype)]
    ring = torch.full((B, max(taps - 1, 1), C), float("nan"), device="cuda")   # nothing of it may be read before it is written
    cache = Cache(cuda, G, D, B, 100, dtype)
    held = [0, 0]
    got_q = [np.zeros((lens[b], H, d)) for b in range(B)]
    table_lens = torch.zeros(B, dtype=torch.int32)
    for s_new, counts in steps:
        counts_b = counts or [s_new] * B
        rows = np.zeros((B, s_new, N))
        for b in range(B):
            rows[b, :counts_b[b]] = u[b][held[b]:held[b] + counts_b[b]]
        for b in range(B):
            table_lens[b] = held[b] + s_new
        # unequal lengths: the cache's own table is per sequence, set through a padded call of the longest, then per row
        _set_lens(cuda, cache, table_lens)
        nl = None if counts is None else torch.tensor(counts, dtype=torch.int32, device="cuda")
        bias, src, acc, gate = None, None, None, None
        if s_new == 1:   # float32 slabs plus the bias
            bias_np = rounded(rng.standard_normal(N), dtype)
            part = rng.standard_normal((2, B, N))
            part[1] = rows[:, 0] - part[0] - bias_np
            acc, bias = dev(part, torch.float32), dev(bias_np, dtype)
            gate = torch.zeros((B, N - C), dtype=convd.dtype, device="cuda")
        else:
            src = dev(rows.reshape(B * s_new, N), dtype)
        q = conv_op(cuda, cache, dtype, src, convd, nd, (H, G), (d, e), B, s_new, ring if taps > 1 else None, D, nl, bias, acc, taps,
                    eps, gate)
        cuda.synchronize()
        qn = q.double().cpu().numpy().reshape(B, s_new, H, D)
        assert (qn[..., d:] == 0).all()
        for b in range(B):
            got_q[b][held[b]:held[b] + counts_b[b]] = qn[b, :counts_b[b], :, :d]
            if gate is not None and counts_b[b]:
                np.testing.assert_allclose(gate[b, :ng].double().cpu().numpy(), rows[b, 0, cols[3]], atol=0.03 if dtype == _lib.BF16 else 1e-5)
            held[b] += counts_b[b]
    assert held == [9, 11]
    for b in range(B):
        assert rms_err(got_q[b].reshape(lens[b], -1), want[b]["q"]) < TOL[dtype]
        for g in range(G):
            k, v = cache.read(b, g, 0, lens[b])
            assert rms_err(k[:, :d], want[b]["k"].reshape(-1, G, d)[:, g]) < TOL[dtype] and (k[:, d:] == 0).all()
            assert rms_err(v[:, :e], want[b]["v"].reshape(-1, G, e)[:, g]) < TOL[dtype] and (v[:, e:] == 0).all()
    cache.close()


def _set_lens(cuda, cache, lens):
    """Per-sequence lengths through the public call: each one in turn, last sequence first."""
    for b in range(len(lens) - 1, -1, -1):
        cache.set_len(b + 1, int(lens[b]))


def attention_case(cuda, dtype, H, G, d, e, base, s_new, window, D, plant=None, B=2, gated=True, alibi=1, scale=0.2, seed=0):
    """(got, want) of the new rows: `base` tokens are cached first, then `s_new` are fed.  plant = (row, distance): that
    query and the key that far behind it are made to stand out, and its value too."""
    rng = np.random.default_rng(seed)
    T = base + s_new
    q, k = rng.standard_normal((B, T, H, d)) * 0.5, rng.standard_normal((B, T, G, d)) * 0.5
    v = rng.standard_normal((B, T, G, e))
    if plant:
        row, dist = plant
        k[:, row - dist] = 3.0
        q[:, row] = 3.0
        v[:, row - dist] = 5.0
    q, k, v = (rounded(a, dtype) for a in (q, k, v))
    gate = rounded(rng.standard_normal((B, T, H * e)), dtype)
    cache = Cache(cuda, G, D, B, T + 3, dtype)
    parts = [(pad8(H * d), q.reshape(B, T, -1)), (pad8(G * d), k.reshape(B, T, -1)), (pad8(G * e), v.reshape(B, T, -1)),
             (pad8(H * e), gate)]
    fused = np.concatenate([np.pad(a, ((0, 0), (0, 0), (0, n - a.shape[2]))) for n, a in parts], axis=2)
    one = torch.ones((1, sum(n for n, _ in parts[:3])), dtype=dev([0], dtype).dtype, device="cuda")
    out = None
    for lo, hi in ((0, base), (base, T)):
        if hi == lo:
            continue
        cache.set_len(B, hi)
        src = dev(fused[:, lo:hi].reshape(B * (hi - lo), -1), dtype)
        qd = conv_op(cuda, cache, dtype, src, one, (None, None), (H, G), (d, e), B, hi - lo, None, D)
        out_ld = pad8(H * e)
        out = torch.zeros((B * (hi - lo), out_ld), dtype=src.dtype, device="cuda")
        g_ptr = ctypes.c_void_p(src.data_ptr() + one.shape[1] * src.element_size()) if gated else None
        _lib.call("rb_attention_window", cuda.ctx, ptr(qd), cache.h, 0, B, hi - lo, H, e, scale, window, alibi, g_ptr,
                  src.shape[1], ptr(out), out_ld, dtype)
        cuda.synchronize()
    cache.close()
    slopes = ref.alibi_slopes(H) if alibi else np.zeros(H)
    want = np.stack([ref.window_attention(q[b], k[b], v[b], scale, slopes, window or T)[base:] for b in range(B)])
    want = want.reshape(B * s_new, H * e)
    if gated:
        want = want * ref.sigmoid(gate[:, base:].reshape(B * s_new, -1))
    return out[:, :H * e].double().cpu().numpy(), want


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,e,D", [(4, 2, 40, 32, 64), (3, 3, 72, 80, 80), (2, 1, 96, 20, 96), (4, 4, 128, 100, 128), (2, 1, 200, 144, 256)])
@pytest.mark.parametrize("base,s_new,window", [(0, 1, 5), (0, 90, 33), (0, 150, 64), (70, 2, 65), (70, 140, 21), (130, 1, 0), (200, 1, 65)])
def test_windowed_attention(cuda, dtype, H, G, d, e, D, base, s_new, window):
    got, want = attention_case(cuda, dtype, H, G, d, e, base, s_new, window, D)
    assert rms_err(got, want) < TOL[dtype] * (1 if dtype == _lib.BF16 else 2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,d", [(64, 48), (96, 96), (128, 104)])
@pytest.mark.parametrize("base,s_new,row", [(0, 160, 159), (0, 160, 128), (0, 100, 99), (64, 130, 193), (191, 1, 191), (192, 1, 192)])
@pytest.mark.parametrize("window", [1, 63, 64, 65])
def test_window_edge_stands_out(cuda, dtype, D, d, base, s_new, row, window):
    """The last key inside the window decides its row; one step further away it must not be seen at all."""
    # no distance bias here, so that the planted score wins by far
    got, want = attention_case(cuda, dtype, 2, 1, d, 16, base, s_new, window, D, plant=(row, window - 1), alibi=0, gated=False)
    assert np.abs(got - want).max() < 0.05
    assert np.abs(want.reshape(2, s_new, -1)[:, row - base] - 5.0).max() < 0.05
    got, want = attention_case(cuda, dtype, 2, 1, d, 16, base, s_new, window, D, plant=(row, window), alibi=0, gated=False)
    assert np.abs(got - want).max() < 0.05
    assert np.abs(got.reshape(2, s_new, -1)[:, row - base] - 5.0).min() > 0.5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("base,s_new", [(0, 300), (299, 1), (100, 200)])
def test_far_key_under_the_distance_bias(cuda, dtype, base, s_new):
    """One key 280 tokens back among small scores, weakest slope: the bias takes 280 / 256 off its score, no more."""
    got, want = attention_case(cuda, dtype, 1, 1, 56, 24, base, s_new, 290, 64, plant=(299, 280), scale=0.05, B=1)
    assert rms_err(got, want) < TOL[dtype] * 2
    assert np.abs(got[-1] - want[-1]).max() < (0.03 if dtype == _lib.BF16 else 1e-4)


@pytest.mark.parametrize("dtype", DTYPES)
def test_many_query_heads_per_key_head(cuda, dtype):
    for base, s_new in ((0, 40), (80, 1)):
        got, want = attention_case(cuda, dtype, 20, 1, 24, 24, base, s_new, 37, 64)
        assert rms_err(got, want) < TOL[dtype] * 2


def hgrn2_op(cuda, cache, dtype, src, f_bias, lower, norm, heads, d, e, batch, s_new, state, chunk=0, new_lens=None, acc=None, eps=1e-4):
    t = src if src is not None else acc
    out_ld = pad8(heads * e)
    out = torch.zeros((batch * s_new, out_ld), dtype=f_bias.dtype, device="cuda")
    _lib.call("rb_hgrn2", cuda.ctx, ptr(src), ptr(acc), 0 if acc is None else acc.shape[0], t.shape[-1], ptr(f_bias), ptr(lower),
              ptr(norm), eps, heads, d, e, batch, s_new, cache.h, ptr(new_lens), ptr(state), chunk, ptr(out), out_ld, dtype)
    cuda.synchronize()
    return out


def hgrn2_want(u, f_bias, lower, norm, H, d, e, eps=1e-4):
    p = pad8(H * d)
    out = np.zeros((u.shape[0], H, e))
    S = []
    for h in range(H):
        c = slice(h * d, (h + 1) * d)
        f = lower[c] + (1 - lower[c]) * ref.sigmoid(u[:, p:2 * p][:, c] + f_bias[c])
        out[:, h], s = ref.gated_linear_recurrence(ref.silu(u[:, c]), f, u[:, 2 * p + h * e:2 * p + (h + 1) * e])
        S.append(s)
    return (ref.rms_normalise(out, eps) * norm).reshape(u.shape[0], -1), np.stack(S)


HGRN_SHAPES = [(3, 32, 48), (2, 72, 24), (2, 128, 128), (2, 20, 36), (1, 13, 30), (1, 130, 140), (2, 64, 256), (1, 256, 256)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,d,e", HGRN_SHAPES)
@pytest.mark.parametrize("chunk", [0, 16, 48])
def test_recurrence(cuda, dtype, H, d, e, chunk):
    """A ragged prompt in pieces, a second portion, then single tokens out of slabs: outputs and the carried state."""
    rng = np.random.default_rng(d + e)
    B, p = 2, pad8(H * d)
    N = 2 * p + pad8(H * e)
    lens = [118, 82]
    steps = [(99, [99, 63]), (17, None), (1, None), (1, None)]
    u = []
    for b in range(B):
        a = rng.standard_normal((lens[b], N))
        a[:, p:2 * p] *= 2
        a[5, p:2 * p] = -120.0   # a token that forgets everything but the lower bound
        a[9, p:2 * p] = 120.0    # and one that takes in nothing
        u.append(rounded(a, dtype))
    f_bias, lower = rounded(rng.uniform(0, 9, H * d), dtype), rounded(np.where(rng.random(H * d) < 0.3, 0, rng.random(H * d)), dtype)
    norm = rounded(1 + 0.2 * rng.standard_normal(e), dtype)
    fd, ld_, nd = dev(f_bias, dtype), dev(lower, dtype), dev(norm, dtype)
    cache = Cache(cuda, 1, 8, B, 200, dtype)
    state = torch.full((B, H, d, e), float("nan"), device="cuda")  # a sequence that starts must not read its slot
    held, got = [0, 0], [[], []]
    for s_new, counts in steps:
        counts_b = counts or [s_new] * B
        rows = np.zeros((B, s_new, N))
        for b in range(B):
            rows[b, :counts_b[b]] = u[b][held[b]:held[b] + counts_b[b]]
            rows[b, counts_b[b]:] = 7.0   # padding that would show
        _set_lens(cuda, cache, [held[b] + s_new for b in range(B)])
        nl = None if counts is None else torch.tensor(counts, dtype=torch.int32, device="cuda")
        if s_new == 1:
            part = rng.standard_normal((3, B, N))
            part[2] = rows[:, 0] - part[0] - part[1]
            out = hgrn2_op(cuda, cache, dtype, None, fd, ld_, nd, H, d, e, B, 1, state, chunk, nl, dev(part, torch.float32))
        else:
            out = hgrn2_op(cuda, cache, dtype, dev(rows.reshape(B * s_new, N), dtype), fd, ld_, nd, H, d, e, B, s_new, state, chunk, nl)
        o = out.double().cpu().numpy().reshape(B, s_new, -1)
        for b in range(B):
            got[b].append(o[b, :counts_b[b], :H * e])
            held[b] += counts_b[b]
    assert held == lens
    for b in range(B):
        want, S = hgrn2_want(u[b], f_bias, lower, norm, H, d, e)
        assert rms_err(np.concatenate(got[b]), want) < (4e-3 if dtype == _lib.BF16 else 1e-5)
        assert rms_err(state[b], S) < 1e-5   # float32 in both dtypes
    cache.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("chunk", [16, 64, 1024, 0])
def test_recurrence_remembers_a_far_token(cuda, chunk, dtype):
    """Gates within 1e-4 of one: a single written token must still be there 900 tokens later, whatever the pieces."""
    H, d, e, T = 1, 48, 40, 1000
    rng = np.random.default_rng(5)
    p = pad8(H * d)
    u = np.zeros((T, 2 * p + pad8(e)))
    u[:, :p] = rng.standard_normal((T, p))
    u[:, 2 * p:] = rng.standard_normal((T, pad8(e))) * 1e-3
    u[:, p:2 * p] = 9.5
    u[60, p:2 * p] = -3.0
    u[60, 2 * p:] = 4.0 * rng.standard_normal(pad8(e))
    u = rounded(u, dtype)
    zero, one = np.zeros(H * d), np.ones(e)
    cache = Cache(cuda, 1, 8, 1, T, dtype)
    cache.set_len(1, T)
    state = torch.zeros((1, H, d, e), device="cuda")
    out = hgrn2_op(cuda, cache, dtype, dev(u, dtype), dev(zero, dtype), dev(zero, dtype), dev(one, dtype), H, d, e, 1, T, state, chunk)
    want, S = hgrn2_want(u, zero, zero, one, H, d, e)
    # the same gate 940 times over: half a float32 ulp of it (3e-8) each time is all that may be lost
    assert rms_err(out[960:], want[960:]) < (4e-3 if dtype == _lib.BF16 else 2e-5)
    assert rms_err(state[0], S) < 4e-5
    cache.close()
