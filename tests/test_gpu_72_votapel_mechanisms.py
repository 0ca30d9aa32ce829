"""Each mechanism of the Votapel design alone, through its C entry point, against the plain oracle."""
import ctypes

import malasun_ref
import numpy as np
import pytest
import torch
import votapel_ref as ref
from malasun_util import DTYPES, TORCH, Cache, dev, pad8, padded, ptr, rms_err, rounded

from rai_b200 import _lib

pytestmark = pytest.mark.gpu
TOL = {_lib.BF16: 6e-3, _lib.F32: 2e-6}


class SharedCache(Cache):
    """A library cache whose values are its keys."""

    def __init__(self, cuda, kv_heads, dim, batch, max_seq, dtype, layers=1):
        self.h = ctypes.c_void_p()
        _lib.call("rb_kv_cache_create_shared", cuda.ctx, layers, kv_heads, dim, batch, max_seq, dtype, ctypes.byref(self.h))
        self.dim, self.dtype = dim, dtype


def zeros(shape, dtype):
    return torch.zeros(shape, dtype=TORCH.get(dtype, dtype), device="cuda")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [52, 320])
def test_embedding_with_positions(cuda, dtype, width):
    """Sequences at different lengths; rows of padding beyond the table are harmless, a token there is reported."""
    rng, ld, B, S, n_pos = np.random.default_rng(width), pad8(width), 3, 7, 40
    table, pos = rounded(rng.standard_normal((77, width)), dtype), rounded(rng.standard_normal((n_pos, width)), dtype)
    ids = rng.integers(0, 77, B * S)
    cache = SharedCache(cuda, 1, 8, B, 64, dtype)
    lens = [7, 30, 45]                       # after this call's rows, padding included
    for b in range(B - 1, -1, -1):
        cache.set_len(b + 1, lens[b])
    new = torch.tensor([7, 5, 2], dtype=torch.int32, device="cuda")   # the third sequence: positions 38, 39, then padding
    td, pd, idd = dev(padded(table, ld), dtype), dev(padded(pos, ld), dtype), torch.from_numpy(ids.astype(np.int32)).cuda()
    h = zeros((B * S, ld), torch.float32)

    def run(new_lens):
        _lib.call("rb_embed_positions", cuda.ctx, ptr(td), ptr(pd), n_pos, dtype, 77, width, ld, ptr(idd), B, S, cache.h, ptr(new_lens), ptr(h))
        cuda.synchronize()
    run(new)
    got = h.double().cpu().numpy()
    for b in range(B):
        for s in range(S):
            p = lens[b] - S + s
            if p < n_pos:
                assert np.abs(got[b * S + s, :width] - (table[ids[b * S + s]] + pos[p])).max() < 1e-6
    assert np.isfinite(got).all() and (got[:, width:] == 0).all()
    with pytest.raises(_lib.RaiB200Error):
        run(None)
    cache.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,rows,top", [(52, 3, 1), (320, 40, 5), (2048, 700, 4), (4104, 33, 2), (9000, 5, 9)])
def test_joint_of_a_block(cuda, dtype, width, rows, top):
    """The stream takes a sublayer's sum (tensor, slabs, weighted experts, or nothing) and the norm of it comes out."""
    rng, ld = np.random.default_rng(width), pad8(width)
    x = rng.standard_normal((rows, width)) * 2
    h = dev(padded(x, ld), torch.float32)
    x = h.double().cpu().numpy()[:, :width]
    gain = rounded(rng.standard_normal(width) * 0.3, dtype)
    y, part = rounded(rng.standard_normal((rows, width)), dtype), rounded(rng.standard_normal((rows * top, width)), dtype)
    slabs, wt = rng.standard_normal((3, rows, width)).astype(np.float32), rng.uniform(0, 2, (rows, top)).astype(np.float32)
    gd, yd, pd = dev(padded(gain[None], ld), dtype), dev(padded(y, ld), dtype), dev(padded(part, ld), dtype)
    sd, wd = dev(np.stack([padded(s, ld) for s in slabs]), torch.float32), dev(wt, torch.float32)
    out = zeros((rows, ld), dtype)
    mixed = (wt[:, :, None] * part.reshape(rows, top, width)).sum(1)
    for tensor, acc, experts, add, mult in ((yd, None, pd, y + mixed, 0.6), (None, sd, pd, slabs.sum(0) + mixed, 1.0),
                                            (None, sd, None, slabs.sum(0), -0.5), (None, None, None, 0 * y, 3.0)):
        _lib.call("rb_add_then_norm", cuda.ctx, ptr(tensor), ptr(acc), 0 if acc is None else 3, ptr(experts),
                  ptr(wd) if experts is not None else None, top, mult, ptr(gd), 0.05, rows, width, ld, ptr(h), ptr(out), dtype)
        x = x + mult * add
        cuda.synchronize()
        assert rms_err(h[:, :width], x) < 1e-6      # the stream is float32 in both dtypes
        assert rms_err(out[:, :width], ref.rms_norm_one_plus(x, gain, 0.05)) < TOL[dtype]
        assert (out[:, width:] == 0).all() and (h[:, width:] == 0).all()
    pick = rng.integers(0, rows, 3)
    few, rd = zeros((3, ld), dtype), torch.from_numpy(pick.astype(np.int32)).cuda()
    _lib.call("rb_one_plus_norm_rows", cuda.ctx, ptr(h), ptr(rd), 0, ptr(gd), 0.05, 3, width, ld, ptr(few), dtype)
    cuda.synchronize()
    assert rms_err(few[:, :width], ref.rms_norm_one_plus(x[pick], gain, 0.05)) < TOL[dtype]


def split(cuda, cache, dtype, fused, H, G, d, F, batch, s_new, slabs=0, bias=None, rng=None):
    """rb_split_append on fused [rows, q | k | gate | up] (numpy, padded parts); returns q and the gated part."""
    D, n = cache.dim, fused.shape[1]
    q, glu = zeros((batch * s_new, H, D), dtype), zeros((batch * s_new, pad8(F) + 16), dtype)
    src = acc = bd = None
    if slabs:
        p = rng.standard_normal((slabs, batch, n))
        p[-1] = fused - p[:-1].sum(0) - bias
        acc, bd = dev(p, torch.float32), dev(bias, dtype)
    else:
        src = dev(fused, dtype)
    _lib.call("rb_split_append", cuda.ctx, ptr(src), ptr(acc), slabs, ptr(bd), n, batch, s_new, H, G, d, F, cache.h, 0, ptr(q),
              ptr(glu) if F else None, glu.shape[1], dtype)
    cuda.synchronize()
    return q, glu


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,D,F", [(4, 2, 40, 64, 56), (3, 1, 20, 64, 33), (6, 6, 64, 64, 0), (5, 5, 13, 80, 8)])
def test_split_and_append(cuda, dtype, H, G, d, D, F):
    """A prompt across a page border, then single tokens out of slabs, at the right places of the cache."""
    rng, B, T = np.random.default_rng(d), 2, 75
    D = pad8(d) if dtype == _lib.F32 else D
    parts = [H * d, G * d, F, F]
    offs = np.cumsum([0] + [pad8(n) for n in parts])
    u = [rounded(rng.standard_normal((B, T, n)), dtype) for n in parts]
    fused = np.zeros((B, T, offs[-1]))
    for a, o in zip(u, offs):
        fused[:, :, o:o + a.shape[2]] = a
    cache = SharedCache(cuda, G, D, B, T + 5, dtype)
    bias = rounded(rng.standard_normal(offs[-1]), dtype)
    at = 0
    for n in (62, 11, 1, 1):
        cache.set_len(B, at + n)
        rows = fused[:, at:at + n].reshape(B * n, -1)
        q, glu = split(cuda, cache, dtype, rows, H, G, d, F, B, n, 3 if n == 1 else 0, bias, rng)
        qn = q.double().cpu().numpy().reshape(B, n, H, D)
        assert rms_err(qn[..., :d], u[0][:, at:at + n].reshape(B, n, H, d)) < TOL[dtype] and (qn[..., d:] == 0).all()
        if F:
            g = glu.double().cpu().numpy()
            want = (ref.silu(u[2]) * u[3])[:, at:at + n].reshape(B * n, F)
            assert rms_err(g[:, :F], want) < TOL[dtype]
            assert (g[:, pad8(F):] == 0).all()
        at += n
    for b in range(B):
        for g in range(G):
            k, v = cache.read(b, g, 0, T)
            assert rms_err(k[:, :d], u[1][b].reshape(T, G, d)[:, g]) < TOL[dtype] and (k[:, d:] == 0).all() and (v == k).all()
    cache.close()


@pytest.mark.parametrize("E,top,groups,keep", [(8, 2, 4, 2), (15, 4, 5, 3), (64, 8, 8, 4), (40, 3, 1, 1), (256, 32, 64, 20), (9, 3, 9, 3),
                                               (48, 1, 2, 1), (5, 5, 1, 1), (96, 6, 3, 1)])
@pytest.mark.parametrize("rows,slabs", [(1, 1), (37, 9), (600, 1)])
def test_routing(cuda, E, top, groups, keep, rows, slabs):
    rng = np.random.default_rng(E + rows)
    ld, cap = E + 11, rows + 3
    z = (rng.standard_normal((slabs, rows, ld)) * (2.0 if slabs == 1 else 0.7)).astype(np.float32)
    if rows > 30:
        z[:, 5] = 0                                  # every score equal: the lower index wins
        z[0, 6, :E] = np.linspace(-9, 30, E)         # scores that round to one
    zd = torch.from_numpy(z).cuda()
    weight, lists, count = zeros((rows, top), torch.float32), torch.full((E, cap), -1, dtype=torch.int32, device="cuda"), zeros(E, torch.int32)
    _lib.call("rb_moe_route", cuda.ctx, ptr(zd), slabs, rows * ld, ld, rows, E, top, groups, keep, 1.7, ptr(weight), ptr(lists), ptr(count), cap)
    cuda.synchronize()
    total = zd[0, :, :E].clone()
    for s in range(1, slabs):
        total += zd[s, :, :E]
    scores = (1.0 / (1.0 + np.exp(-total.cpu().numpy().astype(np.float64)))).astype(np.float32).astype(np.float64)
    count, lists, weight = count.cpu().numpy(), lists.cpu().numpy(), weight.double().cpu().numpy()
    got = {}
    for e in range(E):
        entries = lists[e, :count[e]]
        assert len(set(entries // top)) == count[e] and (lists[e, count[e]:] == -1).all()
        for x in entries:
            got[(x // top, x % top)] = e
    assert len(got) == rows * top
    for r in range(rows):
        want = ref.chosen_experts(scores[r], top, groups, keep)
        mine = [got[(r, j)] for j in range(top)]
        if r != 6 or rows <= 30:                     # (that row's order at the top is a matter of the last bit)
            assert mine == want, r
        np.testing.assert_allclose(weight[r], scores[r, mine] * 1.7, rtol=2e-6)


def routed(rng, rows, E, top, hot=None):
    """Lists of a random routing; `hot` is chosen by every row, expert E - 1 by none."""
    pick = np.stack([rng.permutation(E - 1)[:top] for _ in range(rows)])
    if hot is not None:
        for r in range(rows):
            if hot not in pick[r]:
                pick[r, 0] = hot
    lists, count = np.full((E, rows), -7, dtype=np.int32), np.zeros(E, dtype=np.int32)
    for i in rng.permutation(rows):
        for j in range(top):
            e = pick[i, j]
            lists[e, count[e]] = i * top + j
            count[e] += 1
    return pick, lists, count


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,E,top,W,F", [(1, 4, 2, 72, 40), (9, 12, 3, 136, 200), (40, 6, 2, 256, 136), (150, 200, 3, 64, 72),
                                            (300, 5, 2, 320, 264), (700, 7, 3, 144, 128)])
@pytest.mark.parametrize("with_sorted_copy", [False, True])
def test_expert_products(cuda, dtype, with_sorted_copy, rows, E, top, W, F):
    """Experts with no row, with one, and with more rows than a tile; sizes that are no multiple of any tile."""
    rng = np.random.default_rng(rows)
    pick, lists, count = routed(rng, rows, E, top, hot=1)
    x, wg, wu = (rounded(rng.standard_normal(s) * f, dtype) for s, f in (((rows, W), 1), ((E, F, W), W ** -0.5), ((E, F, W), W ** -0.5)))
    wd = rounded(rng.standard_normal((E, W, F)) * F ** -0.5, dtype)
    xd, gd, ud, dd, ld, cd = dev(x, dtype), dev(wg, dtype), dev(wu, dtype), dev(wd, dtype), torch.from_numpy(lists).cuda(), torch.from_numpy(count).cuda()
    act, out = zeros((rows * top, F), dtype), zeros((rows * top, W), dtype)
    space = zeros((rows * top, W), dtype) if with_sorted_copy else None
    _lib.call("rb_moe_gated", cuda.ctx, ptr(xd), ptr(gd), ptr(ud), ptr(act), rows, top, E, ptr(ld), ptr(cd), rows, F, W, _lib.ACT_SILU,
              ptr(space), dtype)
    _lib.call("rb_moe_down", cuda.ctx, ptr(act), ptr(dd), ptr(out), rows, top, E, ptr(ld), ptr(cd), rows, W, F, dtype)
    cuda.synchronize()
    inner = ref.silu(np.einsum("rw,rjfw->rjf", x, wg[pick])) * np.einsum("rw,rjfw->rjf", x, wu[pick])
    want_act, at = np.zeros((rows * top, F)), 0
    for e in range(E):
        for entry in lists[e, :count[e]]:
            want_act[at] = inner[entry // top, entry % top]
            at += 1
    got_act = act.double().cpu().numpy()
    assert rms_err(got_act, want_act) < TOL[dtype]
    # every row on its own: a row that went astray cannot hide in an average
    row_err = np.sqrt(((got_act - want_act) ** 2).mean(1)) / np.sqrt((want_act ** 2).mean())
    assert row_err.max() < 8 * TOL[dtype]
    want = np.zeros((rows * top, W))
    at = 0
    for e in range(E):
        for entry in lists[e, :count[e]]:
            want[entry] = wd[e] @ got_act[at]
            at += 1
    assert rms_err(out, want) < TOL[dtype]
    assert (np.sqrt(((out.double().cpu().numpy() - want) ** 2).mean(1)) / np.sqrt((want ** 2).mean())).max() < 8 * TOL[dtype]


@pytest.mark.parametrize("rows", [300, 700])
def test_router_logits_of_a_prompt(cuda, rows):
    """One float32 slab for more than 256 rows: the products of bf16 operands without a rounding of the result."""
    rng = np.random.default_rng(rows)
    x, w = rounded(rng.standard_normal((rows, 136)), _lib.BF16), rounded(rng.standard_normal((24, 136)) / 12, _lib.BF16)
    xd, wd, out = dev(x, _lib.BF16), dev(w, _lib.BF16), zeros((rows, 24), torch.float32)
    _lib.call("rb_linear_partials", cuda.ctx, ptr(xd), ptr(wd), ptr(out), rows, 24, 136, 1)
    cuda.synchronize()
    assert rms_err(out, x @ w.T) < 2e-6


def attention_case(cuda, dtype, H, G, d, D, base, s_new, scale=0.2, cap=0.0, sink=None, temp=(0.0, 0), B=2, size=0.5, plant=None, seed=0):
    """(got, want) [B, s_new, H * d]: `base` tokens are cached first, then `s_new` are fed.  plant = (row, key): that query
    and that key are made to stand out."""
    rng = np.random.default_rng(seed)
    T = base + s_new
    q, k = rng.standard_normal((B, T, H, d)) * size, rng.standard_normal((B, T, G, d)) * size
    if plant:
        row, key = plant
        k[:, key] = 3.0
        q[:, row] = 3.0
    q, k = rounded(q, dtype), rounded(k, dtype)
    sink = None if sink is None else rounded(np.broadcast_to(sink, (H,)), dtype)
    D = pad8(d) if dtype == _lib.F32 else D
    cache = SharedCache(cuda, G, D, B, T + 3, dtype)
    fused = np.zeros((B, T, pad8(H * d) + pad8(G * d)))
    fused[:, :, :H * d] = q.reshape(B, T, -1)
    fused[:, :, pad8(H * d):pad8(H * d) + G * d] = k.reshape(B, T, -1)
    out_ld = pad8(H * d) + 8
    sd = None if sink is None else dev(sink, dtype)
    o = _lib.AttentionOptions(temp_every=temp[1], temp_coef=temp[0], softcap=cap, value_dim=d, sink=ptr(sd), out_ld=out_ld)
    out = None
    for lo, hi in ((0, base), (base, T)):
        if hi == lo:
            continue
        cache.set_len(B, hi)
        qd, _ = split(cuda, cache, dtype, fused[:, lo:hi].reshape(B * (hi - lo), -1), H, G, d, 0, B, hi - lo)
        out = zeros((B * (hi - lo), out_ld), dtype)
        _lib.call("rb_attention_general", cuda.ctx, ptr(qd), cache.h, 0, B, hi - lo, H, scale, ctypes.byref(o), ptr(out), dtype)
        cuda.synchronize()
    cache.close()
    assert (out[:, H * d:] == 0).all()
    warm = np.array([ref.query_temperature(p, *temp) if temp[1] else 1.0 for p in range(T)]).reshape(T, 1, 1)
    want = [ref.attention((q[b] * warm)[base:], k[b], k[b], scale, cap, np.full(H, -1e30) if sink is None else sink, base) for b in range(B)]
    return out[:, :H * d].double().cpu().numpy().reshape(B, s_new, H * d), np.stack(want).reshape(B, s_new, H * d)


SHAPES = [(4, 2, 40, 64), (3, 3, 72, 80), (6, 1, 96, 96), (4, 4, 100, 128), (8, 1, 64, 64), (2, 1, 128, 128), (2, 1, 200, 256)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,D", SHAPES)
@pytest.mark.parametrize("base,s_new", [(0, 1), (0, 90), (0, 150), (70, 2), (70, 140), (130, 1), (300, 1)])
def test_attention_with_everything(cuda, dtype, H, G, d, D, base, s_new):
    got, want = attention_case(cuda, dtype, H, G, d, D, base, s_new, cap=2.5, sink=np.linspace(-1, 3, H), temp=(0.7, 9))
    assert rms_err(got, want) < TOL[dtype] * 2


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,d", [(64, 56), (96, 96), (128, 128)])
@pytest.mark.parametrize("base,s_new", [(0, 140), (0, 60), (128, 1)])
@pytest.mark.parametrize("what", ["cap, scores far below it", "cap, scores around it", "cap, scores far above it", "sink", "temperature", "plain"])
def test_attention_one_thing_at_a_time(cuda, dtype, D, d, base, s_new, what):
    kw = {"cap, scores far below it": dict(cap=30.0, size=0.5), "cap, scores around it": dict(cap=3.0, size=1.0),
          "cap, scores far above it": dict(cap=1.5, size=2.5), "sink": dict(sink=[-2.0, 0.0, 2.0, 6.0]),
          "temperature": dict(temp=(1.5, 16)), "plain": {}}[what]
    got, want = attention_case(cuda, dtype, 4, 2, d, D, base, s_new, **kw)
    assert rms_err(got, want) < TOL[dtype] * 2


@pytest.mark.parametrize("dtype", DTYPES)
def test_cap_is_exact_in_both_forms(cuda, dtype):
    """A large cap multiplies whatever error the capped score has: scores up to 40 under a cap of 100, and up to 90."""
    for size in (0.8, 1.25):
        got, want = attention_case(cuda, dtype, 2, 2, 64, 64, 0, 130, scale=0.8, cap=100.0, size=size)
        assert rms_err(got, want) < TOL[dtype] * 2


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,d", [(64, 48), (96, 96), (128, 104)])
@pytest.mark.parametrize("base,s_new,row", [(0, 330, 329), (0, 330, 128), (0, 100, 99), (256, 130, 385), (319, 1, 319), (320, 1, 320), (321, 2, 322)])
@pytest.mark.parametrize("key", [0, 1, 63, 64, "row"])
def test_a_far_key_stands_out(cuda, dtype, D, d, base, s_new, row, key):
    """One key among hundreds, at the very start, at page borders, or the row's own: it decides the row under the cap."""
    key = row if key == "row" else key
    got, want = attention_case(cuda, dtype, 2, 1, d, D, base, s_new, cap=14.0, plant=(row, key), sink=1.0)
    assert np.abs(got - want).max() < 0.05
    assert np.abs(want[:, row - base] - 3.0).max() < 0.2      # (the oracle: the key did decide the row)
    if key < row:                                     # nor is it seen before its time
        got, want = attention_case(cuda, dtype, 2, 1, d, D, base, s_new, cap=14.0, plant=(row - 1 if row > base else row, row), sink=1.0)
        assert np.abs(got - want).max() < 0.05


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("base,s_new", [(0, 1), (0, 40), (0, 200), (700, 1), (200, 3)])
def test_sinks_small_and_overwhelming(cuda, dtype, base, s_new):
    """A sink next to nothing, one as heavy as all keys together, and one so heavy that exp of it overflows a float."""
    got, want = attention_case(cuda, dtype, 4, 2, 64, 64, base, s_new, sink=[-60.0, 5.5, 20.0, 200.0])
    assert rms_err(got, want) < TOL[dtype] * 2
    assert np.abs(got[..., 192:]).max() == 0 and np.abs(got[..., 128:192]).max() < 1e-4
    light, _ = attention_case(cuda, dtype, 4, 2, 64, 64, base, s_new, sink=None)
    assert rms_err(light[..., :64], got[..., :64]) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("base", [6, 7, 8, 127, 128])
def test_temperature_edges(cuda, dtype, base):
    """Around a multiple of the stretch; a large coefficient makes one step of it visible."""
    got, want = attention_case(cuda, dtype, 2, 1, 64, 64, base, 1, temp=(4.0, 8), scale=0.3)
    assert rms_err(got, want) < TOL[dtype] * 2
    got, want = attention_case(cuda, dtype, 2, 1, 64, 64, 0, base + 20, temp=(4.0, 8), scale=0.3)
    assert rms_err(got, want) < TOL[dtype] * 2


@pytest.mark.parametrize("dtype", DTYPES)
def test_many_query_heads_per_key_head(cuda, dtype):
    for base, s_new in ((0, 40), (80, 1)):
        got, want = attention_case(cuda, dtype, 20, 1, 24, 64, base, s_new, cap=2.0, sink=np.linspace(-1, 1, 20), temp=(0.5, 11))
        assert rms_err(got, want) < TOL[dtype] * 2


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D", [64, 96])
@pytest.mark.parametrize("T,s_new", [(150, 150), (70, 70), (90, 1)])
def test_cap_and_sink_beside_window_bias_and_separate_values(cuda, dtype, D, T, s_new):
    """The options combine: a rolling window and the distance bias over a cache with values of its own."""
    rng = np.random.default_rng(D)
    H, G, window, cap, scale, sink = 4, 2, 37, 1.5, 0.3, rounded([0.5, -1.0, 2.0, 0.0], dtype)
    q, k, v = (rounded(rng.standard_normal(s), dtype) for s in ((T, H, D), (T, G, D), (T, G, D)))
    cache = Cache(cuda, G, D, 1, T + 1, dtype)
    one = torch.ones((1, (H + 2 * G) * D), dtype=TORCH[dtype], device="cuda")
    sd = dev(sink, dtype)
    o = _lib.AttentionOptions(window=window, alibi=1, softcap=cap, sink=ptr(sd), value_dim=D, out_ld=H * D)
    for lo, hi in ((0, T - s_new), (T - s_new, T)):
        if lo == hi:
            continue
        cache.set_len(1, hi)
        src = dev(np.concatenate([a[lo:hi].reshape(hi - lo, -1) for a in (q, k, v)], axis=1), dtype)
        qd, out = zeros((hi - lo, H, D), dtype), zeros((hi - lo, H * D), dtype)
        _lib.call("rb_conv_norm_append", cuda.ctx, ptr(src), None, 0, None, ptr(one), 1, None, None, 1e-6, 1, hi - lo, H, G, D, D,
                  src.shape[1], cache.h, 0, None, None, ptr(qd), None, dtype)
        _lib.call("rb_attention_general", cuda.ctx, ptr(qd), cache.h, 0, 1, hi - lo, H, scale, ctypes.byref(o), ptr(out), dtype)
        cuda.synchronize()
    cache.close()
    slopes = malasun_ref.alibi_slopes(H)
    want = np.zeros((s_new, H, D))
    for h in range(H):
        for r in range(s_new):
            i = T - s_new + r
            lo = max(0, i - window + 1)
            s = ref.soft_cap(k[lo:i + 1, h // 2] @ q[i, h] * scale, cap) - slopes[h] * (i - np.arange(lo, i + 1))
            want[r, h] = ref.sink_softmax(s, sink[h]) @ v[lo:i + 1, h // 2]
    assert rms_err(out, want.reshape(s_new, -1)) < TOL[dtype] * 2
