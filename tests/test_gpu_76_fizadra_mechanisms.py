"""Each mechanism of the Fizadra design alone, through its C entry point, against the plain oracle."""
import ctypes

import fizadra_ref as ref
import numpy as np
import pytest
import torch
from malasun_util import DTYPES, TORCH, Cache, dev, pad8, padded, ptr, rms_err, rounded

from rai_b200 import _lib
from rai_b200.configs import yarn_rotation

pytestmark = pytest.mark.gpu
TOL = {_lib.BF16: 6e-3, _lib.F32: 2e-6}


def zeros(shape, dtype):
    return torch.zeros(shape, dtype=TORCH.get(dtype, dtype), device="cuda")


def slabs_of(rng, total, n):
    """n float32 arrays that sum to `total` up to rounding."""
    p = rng.standard_normal((n,) + total.shape)
    p[-1] = total - p[:-1].sum(0)
    return dev(p, torch.float32)


def weight(rng, n, dtype):
    return rounded(1 + 0.3 * rng.standard_normal(n), dtype)


def dev_weight(w, dtype):
    return dev(np.pad(w, (0, pad8(len(w)) - len(w))), dtype)


class LatentCache(Cache):
    """A cache whose values are its keys, one head."""

    def __init__(self, cuda, dim, batch, max_seq, dtype, layers=1):
        self.h = ctypes.c_void_p()
        _lib.call("rb_kv_cache_create_shared", cuda.ctx, layers, 1, dim, batch, max_seq, dtype, ctypes.byref(self.h))
        self.dim, self.dtype = dim, dtype


# ---- joints and norms

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,groups,rows", [(52, 1, 3), (52, 4, 5), (96, 3, 40), (512, 2, 33), (1024, 4, 700), (1024, 8, 3), (4096, 2, 9), (4104, 3, 6),
                                               (6144, 24, 4), (75, 25, 11)])
@pytest.mark.parametrize("slabs", [0, 1, 9])
def test_joint(cuda, dtype, width, groups, rows, slabs):
    rng, ld, eps = np.random.default_rng(width + groups), pad8(width), 0.03
    gains = [weight(rng, width, dtype) for _ in range(2)]
    h = np.asarray(rng.standard_normal((rows, width)) * 2, dtype=np.float32).astype(np.float64)
    y = rounded(rng.standard_normal((rows, width)) * np.repeat(rng.uniform(0.1, 3, groups), width // groups), dtype)
    src = acc = None
    if slabs:
        acc = slabs_of(rng, padded(y, ld), slabs)
        acc[:, :, width:] = 0
        y = acc.double().sum(0).cpu().numpy()[:, :width]
    else:
        src = dev(padded(y, ld), dtype)
    hd, pd, gd, out = dev(padded(h, ld), torch.float32), dev_weight(gains[0], dtype), dev_weight(gains[1], dtype), zeros((rows, ld), dtype)
    _lib.call("rb_sandwich_join", cuda.ctx, ptr(src), ptr(acc), slabs, ptr(pd), groups, eps, rows, width, ld, ptr(hd), ptr(hd), None, 0, None, 0,
              ptr(gd), ptr(out), dtype)
    cuda.synchronize()
    x = h + ref.group_norm(y, gains[0], groups, eps)
    assert rms_err(hd[:, :width], x) < 1e-6                       # float32 in both dtypes
    assert rms_err(out[:, :width], ref.group_norm(x, gains[1], groups, eps)) < TOL[dtype]
    assert (out[:, width:] == 0).all() and (hd[:, width:] == 0).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,groups,n", [(72, 3, 2), (512, 1, 3), (1024, 4, 9), (100, 5, 17)])
def test_depth_average(cuda, dtype, width, groups, n):
    """The result joins a history of n - 1 others; without a norm behind it, and once more from the history's first entry."""
    rng, ld, rows, eps = np.random.default_rng(n), pad8(width), 21, 0.02
    hist = np.asarray(rng.standard_normal((n, rows, width)), dtype=np.float32).astype(np.float64)
    wts, post = rounded(rng.standard_normal(n), dtype), weight(rng, width, dtype)
    y, h = rounded(rng.standard_normal((rows, width)), dtype), hist[0]
    room = rows * ld + 8 * ld                                     # (a history may hold more rows than this call)
    hd = zeros((n, room), torch.float32)
    hd[:, :rows * ld] = dev(np.stack([padded(a, ld).ravel() for a in hist]), torch.float32)
    hd[n - 1] = float("nan")
    yd, pd, wd, out = dev(padded(y, ld), dtype), dev_weight(post, dtype), dev_weight(wts, dtype), zeros((rows, ld), torch.float32)
    _lib.call("rb_sandwich_join", cuda.ctx, ptr(yd), None, 0, ptr(pd), groups, eps, rows, width, ld, ptr(hd), ptr(out), ptr(wd), n, ptr(hd), room,
              None, None, dtype)
    cuda.synchronize()
    x = h + ref.group_norm(y, post, groups, eps)
    got = hd[:, :rows * ld].reshape(n, rows, ld)
    assert rms_err(got[n - 1, :, :width], x) < 1e-6
    assert rms_err(out[:, :width], ref.depth_average(wts, list(hist[:-1]) + [x])) < 1e-6
    assert rms_err(got[:-1, :, :width], hist[:-1]) == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,groups", [(60, 5), (1024, 4), (72, 1), (4104, 4)])
def test_norm_of_chosen_rows(cuda, dtype, width, groups):
    rng, ld = np.random.default_rng(width), pad8(width)
    h, gain = np.asarray(rng.standard_normal((24, width)), dtype=np.float32).astype(np.float64), weight(rng, width, dtype)
    hd, gd = dev(padded(h, ld), torch.float32), dev_weight(gain, dtype)
    for rows, step, want in ((np.array([7, 0, 23, 7]), 0, [7, 0, 23, 7]), (None, 6, [5, 11, 17, 23])):
        rd = None if rows is None else torch.from_numpy(rows.astype(np.int32)).cuda()
        out = zeros((4, ld), dtype)
        _lib.call("rb_group_norm_rows", cuda.ctx, ptr(hd), ptr(rd), step, ptr(gd), groups, 0.05, 4, width, ld, ptr(out), dtype)
        cuda.synchronize()
        assert rms_err(out[:, :width], ref.group_norm(h[want], gain, groups, 0.05)) < TOL[dtype] and (out[:, width:] == 0).all()


# ---- rotation

def tables(cuda, rot, n):
    cos, sin = (torch.empty((n, rot["dims"] // 2), device="cuda") for _ in range(2))
    s = rot["scaling"]
    if s:
        _lib.call("rb_rotary_tables_yarn", cuda.ctx, rot["dims"], n, rot["base"], s["factor"], s["fast"], s["slow"], s["original"], ptr(cos), ptr(sin))
    else:
        _lib.call("rb_rotary_tables", cuda.ctx, rot["dims"], n, rot["base"], 1.0, 1.0, 1.0, 0.0, ptr(cos), ptr(sin))
    return cos, sin


@pytest.mark.parametrize("rot", [yarn_rotation(64, 1e4, 8.0, 32.0, 1.0, 512), yarn_rotation(6, 50.0, 3.0, 4.0, 0.5, 40), yarn_rotation(16, 700.0, 5.0, 9.0, 0.5, 90),
                                 yarn_rotation(2, 9.0, 2.0, 2.0, 1.0, 8), yarn_rotation(32, 1e4, 4.0, 2.0, 2.0, 100), yarn_rotation(24, 1e3, 40.0, 1e6, 1e-9, 64)])
def test_yarn_tables(cuda, rot):
    cos, sin = tables(cuda, rot, 3000)
    a, amp = np.arange(3000)[:, None] * np.array(ref.rotary_frequencies(rot)), ref.rotary_amplitude(rot)
    assert amp > 1
    assert np.abs(cos.cpu().numpy() - amp * np.cos(a)).max() < 2e-6 and np.abs(sin.cpu().numpy() - amp * np.sin(a)).max() < 2e-6


# ---- what surrounds latent attention

LATENTS = [  # q_rank, kv_rank, rot_dim, turning, interleaved
    (40, 72, 16, 16, True), (56, 64, 32, 32, False), (33, 45, 6, 6, True), (33, 45, 10, 10, False), (64, 512, 64, 64, True), (1536, 128, 24, 16, False),
    (8, 8, 0, 0, False), (17, 100, 28, 20, True)]


def latent_dim(dtype, kv_rank, rot_dim):
    n = pad8(kv_rank) + rot_dim
    return (n + 63) // 64 * 64 if dtype == _lib.BF16 else pad8(n)


def rotation_of(turning, interleaved):
    return yarn_rotation(turning, 1e3, 4.0, 8.0, 0.5, 128, interleaved) if turning else None


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("qr,kr,rd,turning,interleaved", LATENTS)
@pytest.mark.parametrize("gate", [0, 5, 300])
def test_norms_rotation_append_and_gather(cuda, dtype, qr, kr, rd, turning, interleaved, gate):
    """A prompt across a page border, portions, single tokens out of slabs, at the right places of the cache; then the same
    latents out of the cache, and a projection without a latent of its own."""
    rng, B, T, eps = np.random.default_rng(qr + kr), 2, 150, 0.02
    rot = rotation_of(turning, interleaved)
    offs = np.cumsum([0, pad8(qr), pad8(kr + rd), pad8(gate)])
    u = [rounded(rng.standard_normal((B, T, n)) * 2, dtype) for n in (qr, kr + rd, gate)]
    fused = np.zeros((B, T, offs[-1]))
    for a, o in zip(u, offs):
        fused[:, :, o:o + a.shape[2]] = a
    qw, kw = weight(rng, qr, dtype), weight(rng, kr, dtype)
    qd, kd = dev_weight(qw, dtype), dev_weight(kw, dtype)
    cache = LatentCache(cuda, latent_dim(dtype, kr, rd), B, T + 5, dtype)
    cos, sin = tables(cuda, rot, T + 70) if rot else (None, None)
    want_q = ref.rms(u[0], eps) * qw
    want = np.concatenate([ref.rms(u[1][..., :kr], eps) * kw, np.stack([ref.rotate(u[1][b, :, None, kr:], rot)[:, 0] for b in range(B)])], -1)
    at = 0
    for n in (62, 11, 1, 74, 1, 1):
        cache.set_len(B, at + n)
        rows = B * n
        part = fused[:, at:at + n].reshape(rows, -1)
        slabs = 7 if n == 1 and at > 80 else 0
        src, acc = (None, slabs_of(rng, part, slabs)) if slabs else (dev(part, dtype), None)
        if slabs:
            for o, w in zip(offs, (qr, kr + rd, gate)):
                acc[:, :, o + w:o + pad8(w)] = 0
        cq, lat = zeros((rows, pad8(qr)), dtype), zeros((rows, pad8(kr)), dtype)
        g = torch.full((rows, pad8(max(gate, 1))), 9.0, dtype=TORCH[dtype], device="cuda") if gate else None
        _lib.call("rb_latent_append", cuda.ctx, ptr(src), ptr(acc), slabs, fused.shape[2], qr, kr, rd, ptr(qd), ptr(kd), eps, ptr(cos), ptr(sin), turning,
                  int(interleaved), B, n, cache.h, 0, ptr(cq), ptr(lat), ptr(g), gate, dtype)
        back, alone = zeros((rows, pad8(kr)), dtype), zeros((rows, pad8(qr)), dtype)
        _lib.call("rb_latent_gather", cuda.ctx, cache.h, 0, kr, B, n, ptr(back), dtype)
        own = dev(np.delete(part, np.s_[offs[1]:offs[2]], 1), dtype)
        _lib.call("rb_latent_append", cuda.ctx, ptr(own), None, 0, own.shape[1], qr, 0, rd, ptr(qd), None, eps, ptr(cos), ptr(sin), turning, int(interleaved),
                  B, n, cache.h, 0, ptr(alone), None, None, 0, dtype)
        cuda.synchronize()
        assert rms_err(cq[:, :qr], want_q[:, at:at + n].reshape(rows, qr)) < TOL[dtype] and (cq[:, qr:] == 0).all()
        assert rms_err(alone, cq.double().cpu().numpy()) < TOL[dtype]
        assert rms_err(lat[:, :kr], want[:, at:at + n, :kr].reshape(rows, kr)) < TOL[dtype]
        assert torch.equal(lat, back) and (lat[:, kr:] == 0).all()
        if gate:
            assert rms_err(g[:, :gate], u[2][:, at:at + n].reshape(rows, gate)) < TOL[dtype]
        at += n
    for b in range(B):
        k, _ = cache.read(b, 0, 0, T)
        assert rms_err(k[:, :kr], want[b, :, :kr]) < TOL[dtype] and (rd == 0 or rms_err(k[:, kr:kr + rd], want[b, :, kr:]) < TOL[dtype])
        assert (k[:, kr + rd:] == 0).all()
    cache.close()


def fill_latents(cuda, cache, rng, dtype, B, T, kr, rd, loud=None):
    """Random latents and key parts in the cache, as the cache holds them [B, T, kr + rd].  loud = (token, factor)."""
    u = rng.standard_normal((B, T, kr + rd))
    if loud:
        u[:, loud[0]] = loud[1]
    fused = np.zeros((B, T, 8 + pad8(kr + rd)))
    fused[:, :, :8] = 1
    fused[:, :, 8:8 + kr + rd] = rounded(u, dtype)
    one, kw, cq = dev(np.ones(8), dtype), dev(np.ones(pad8(kr)), dtype), zeros((B * T, 8), dtype)
    src = dev(fused.reshape(B * T, -1), dtype)
    cache.set_len(B, T)
    _lib.call("rb_latent_append", cuda.ctx, ptr(src), None, 0, fused.shape[2], 8, kr, rd, ptr(one), ptr(kw), 1e-5, None, None, 0, 0, B, T, cache.h, 0, ptr(cq),
              None, None, 0, dtype)
    cuda.synchronize()
    return np.stack([cache.read(b, 0, 0, T)[0][:, :kr + rd] for b in range(B)])


PRODUCTS = [  # heads, dim, rot_dim, turning, interleaved, kv_rank, vdim
    (4, 32, 16, 16, True, 72, 40), (3, 24, 8, 8, False, 64, 24), (5, 13, 6, 6, True, 45, 20), (2, 96, 32, 32, False, 512, 128), (16, 64, 64, 64, True, 128, 64),
    (1, 20, 0, 0, False, 200, 7), (2, 128, 64, 40, False, 600, 200)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,d,rd,turning,interleaved,kr,e", PRODUCTS)
@pytest.mark.parametrize("batch,s_new,slabs", [(3, 1, 0), (3, 1, 6), (1, 70, 0), (2, 33, 0), (70, 1, 3)])
def test_into_the_latents_space_and_out(cuda, dtype, H, d, rd, turning, interleaved, kr, e, batch, s_new, slabs):
    rng, rows, at = np.random.default_rng(H * d), batch * s_new, 41
    rot = rotation_of(turning, interleaved)
    cache = LatentCache(cuda, latent_dim(dtype, kr, rd), batch, at + s_new, dtype)
    cache.set_len(batch, at + s_new)
    cos, sin = tables(cuda, rot, 192) if rot else (None, None)
    q = rounded(rng.standard_normal((batch, s_new, H, d + rd)), dtype)
    uk, uv = (rounded(rng.standard_normal((H, n, kr)) / np.sqrt(n if n == d else kr), dtype) for n in (d, e))
    ld, kp = pad8(H * (d + rd)) + 8, pad8(kr)
    flat = padded(q.reshape(rows, -1), ld)
    src, acc = (None, slabs_of(rng, flat, slabs)) if slabs else (dev(flat, dtype), None)
    stack = lambda a: dev(np.pad(a, ((0, 0), (0, 0), (0, kp - kr))).reshape(-1, kp), dtype)  # noqa: E731
    ukd, uvd = stack(uk), stack(uv)
    out = torch.full((rows, H, cache.dim), 9.0, dtype=TORCH[dtype], device="cuda")
    _lib.call("rb_latent_query", cuda.ctx, ptr(src), ptr(acc), slabs, ld, ptr(ukd), H, d, rd, kr, ptr(cos), ptr(sin), turning, int(interleaved), batch, s_new,
              cache.h, ptr(out), dtype)
    cuda.synchronize()
    want = np.einsum("bshd,hdr->bshr", q[..., :d], uk)
    turned = np.stack([ref.rotate(q[b, :, :, d:], rot, at) for b in range(batch)])
    got = out.double().cpu().numpy().reshape(batch, s_new, H, -1)
    assert rms_err(got[..., :kr], want) < TOL[dtype] and (rd == 0 or rms_err(got[..., kr:kr + rd], turned) < TOL[dtype])
    assert (got[..., kr + rd:] == 0).all()
    x = rounded(rng.standard_normal((rows, H, kr)), dtype)
    xd = dev(np.pad(x, ((0, 0), (0, 0), (0, kp - kr))).reshape(rows, -1), dtype)
    for per_head in (None, False, True):
        n = H if per_head else H * e
        gate = rounded(rng.standard_normal((rows, n)) * 2, dtype)
        gd, o = dev(padded(gate, pad8(n) + 8), dtype), zeros((rows, pad8(H * e) + 8), dtype)
        _lib.call("rb_latent_output", cuda.ctx, ptr(xd), ptr(uvd), H, kr, e, None if per_head is None else ptr(gd), pad8(n) + 8, int(bool(per_head)), rows,
                  ptr(o), pad8(H * e) + 8, dtype)
        cuda.synchronize()
        w = np.einsum("rhk,hek->rhe", x, uv)
        if per_head is not None:
            w = w * ref.sigmoid(gate.reshape(rows, H, 1) if per_head else gate.reshape(rows, H, e))
        assert rms_err(o[:, :H * e], w.reshape(rows, -1)) < TOL[dtype] and (o[:, H * e:] == 0).all()
    cache.close()


# ---- attention

def talking_case(cuda, dtype, H, G, d, e, base, s_new, scale=0.2, B=2, sink=None, plant=None, seed=0, window=0, chunk=0,
                 on_host=True):
    """(got, want) [B, s_new, H, e]: `base` tokens are cached, `s_new` are fed.  plant = (row, key): that query's and that key's
    scores stand out after mixing, and the key's value is 5."""
    rng, T = np.random.default_rng(seed), base + s_new
    q, k, v = (rng.standard_normal((B, T) + n) * 0.5 for n in ((H, d), (G, d), (G, e)))
    talk = rounded(np.eye(H) + rng.standard_normal((H, H)) / np.sqrt(H), dtype)
    if plant:
        row, key = plant
        talk = rounded(np.abs(talk), dtype)
        q[:, row], k[:, key], v[:, key] = 3.0, 3.0, 5.0
    q, k, v = (rounded(a, dtype) for a in (q, k, v))
    widest = max(d, e)
    cache = Cache(cuda, G, (widest + 63) // 64 * 64 if dtype == _lib.BF16 else pad8(widest), B, T + 3, dtype)
    offs = np.cumsum([0, pad8(H * d), pad8(G * d), pad8(G * e)])
    fused = np.zeros((B, T, offs[-1]))
    for a, o in zip((q, k, v), offs):
        fused[:, :, o:o + a[0, 0].size] = a.reshape(B, T, -1)
    host = np.ascontiguousarray(talk, dtype=np.float32)
    td, sd, out_ld = dev(talk, dtype), None if sink is None else dev(sink, dtype), pad8(H * e) + 8
    for lo, hi in ((0, base), (base, T)):
        if hi == lo:
            continue
        n = B * (hi - lo)
        cache.set_len(B, hi)
        src, qd, out = dev(fused[:, lo:hi].reshape(n, -1), dtype), zeros((n, H, cache.dim), dtype), zeros((n, out_ld), dtype)
        _lib.call("rb_head_norm_rope_append", cuda.ctx, ptr(src), None, 0, None, fused.shape[2], None, None, 1e-5, None, None, 0, B, hi - lo, H, G, d, e,
                  cache.h, 0, ptr(qd), None, 0, dtype)
        if lo == base:
            o = _lib.AttentionOptions(value_dim=e, out_ld=out_ld, talk=ptr(td), sink=ptr(sd), window=window, chunk=chunk,
                                      talk_host=host.ctypes.data if on_host else None)
            _lib.call("rb_attention_general", cuda.ctx, ptr(qd), cache.h, 0, B, hi - lo, H, scale, ctypes.byref(o), ptr(out), dtype)
        cuda.synchronize()
    cache.close()
    assert (out[:, H * e:] == 0).all()
    return out[:, :H * e].double().cpu().numpy().reshape(B, s_new, H, e), (q, k, v, talk)


def rounded_sink(rng, H, dtype):
    return rounded(rng.standard_normal(H) * 2, dtype)


TALKS = [(4, 2, 40, 24), (3, 3, 72, 80), (6, 1, 96, 56), (8, 8, 96, 128), (9, 3, 20, 13), (16, 4, 128, 64), (12, 12, 64, 64), (4, 2, 200, 160), (6, 6, 64, 200),
         (2, 1, 256, 40), (24, 24, 32, 32), (1, 1, 64, 64), (40, 2, 32, 32), (32, 8, 128, 128), (10, 10, 136, 136), (20, 20, 64, 144), (36, 36, 24, 16),
         (32, 32, 128, 128), (16, 16, 128, 64), (12, 12, 128, 128), (8, 8, 128, 128), (7, 7, 200, 256), (12, 3, 96, 96), (5, 5, 64, 64), (24, 8, 64, 32)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,e", TALKS)
@pytest.mark.parametrize("base,s_new", [(0, 1), (0, 2), (0, 70), (33, 2), (70, 45), (130, 1), (230, 9), (300, 1)])
def test_attention_with_mixed_heads(cuda, dtype, H, G, d, e, base, s_new):
    sink = rounded_sink(np.random.default_rng(H), H, dtype)
    got, (q, k, v, talk) = talking_case(cuda, dtype, H, G, d, e, base, s_new, sink=sink)
    want = np.stack([ref.attention(q[b, base:], k[b], v[b], 0.2, sink, talk, base) for b in range(2)])
    assert rms_err(got, want) < TOL[dtype]


@pytest.mark.parametrize("H,G,d,e", [(8, 4, 64, 64), (16, 16, 128, 128), (5, 1, 128, 64)])
@pytest.mark.parametrize("base,s_new", [(0, 70), (70, 45)])
def test_mixing_known_on_the_device_only(cuda, H, G, d, e, base, s_new):
    got, (q, k, v, talk) = talking_case(cuda, _lib.BF16, H, G, d, e, base, s_new, on_host=False)
    want = np.stack([ref.attention(q[b, base:], k[b], v[b], 0.2, None, talk, base) for b in range(2)])
    assert rms_err(got, want) < TOL[_lib.BF16]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,e", [(8, 8, 96, 128), (16, 4, 128, 64), (6, 1, 96, 56)])
@pytest.mark.parametrize("base,s_new", [(0, 300), (999, 1), (700, 1), (301, 64)])
def test_attention_with_mixed_heads_at_length(cuda, dtype, H, G, d, e, base, s_new):
    """Several blocks of a prompt; single tokens whose keys are shared out over blocks."""
    got, (q, k, v, talk) = talking_case(cuda, dtype, H, G, d, e, base, s_new, B=1, sink=np.zeros(H), seed=5)
    rows = list(range(s_new))[::29] + [s_new - 1]
    want = np.stack([ref.attention(q[0, base + i:base + i + 1], k[0], v[0], 0.2, np.zeros(H), talk, base + i)[0] for i in rows])
    assert rms_err(got[0, rows], want) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("row,key", [(64, 0), (64, 63), (65, 64), (127, 0), (128, 127), (128, 128), (31, 31), (32, 31), (33, 32), (190, 3), (190, 95), (190, 96)])
@pytest.mark.parametrize("single", [False, True])
def test_one_key_stands_out_for_mixed_heads(cuda, dtype, row, key, single):
    """At page and tile borders, first and last: the row that looks for the key gets its value, the row before the key nothing."""
    H, G, d, e = 6, 3, 40, 24
    base, s_new = (row, 1) if single else (0, 191)
    got, (q, k, v, talk) = talking_case(cuda, dtype, H, G, d, e, base, s_new, plant=(row, key), seed=row)
    want = np.stack([ref.attention(q[b, base:], k[b], v[b], 0.2, None, talk, base) for b in range(2)])
    assert rms_err(got, want) < 2 * TOL[dtype]
    assert np.abs(got[:, row - base] - 5.0).max() < 0.05


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,chunk", [(1, 0), (32, 0), (50, 0), (64, 0), (0, 33), (0, 64), (40, 50)])
@pytest.mark.parametrize("base,s_new", [(0, 140), (139, 1), (70, 20)])
def test_mixed_heads_in_windows_and_chunks(cuda, dtype, window, chunk, base, s_new):
    """Options this design does not set."""
    H, G, d, e = 4, 2, 40, 24
    got, (q, k, v, talk) = talking_case(cuda, dtype, H, G, d, e, base, s_new, window=window, chunk=chunk)
    for b in range(2):
        for i in range(0, s_new, 7):
            p = base + i
            lo = max(0, p - window + 1 if window else 0, p // chunk * chunk if chunk else 0)
            want = ref.attention(q[b, p:p + 1], k[b, lo:p + 1], v[b, lo:p + 1], 0.2, None, talk, p - lo)[0]
            assert rms_err(got[b, i], want) < 2 * TOL[dtype], (b, i)


def latent_case(cuda, dtype, H, kr, rd, base, s_new, scale=0.1, B=2, sink=None, loud=None, seed=0):
    """(got, want) [B, s_new, H, kr] of attention over latents that are in the cache already."""
    rng, T = np.random.default_rng(seed), base + s_new
    cache = LatentCache(cuda, latent_dim(dtype, kr, rd), B, T + 3, dtype)
    c = fill_latents(cuda, cache, rng, dtype, B, T, kr, rd, loud)
    q = rng.standard_normal((B, s_new, H, kr + rd)) * 0.4
    if loud:
        q[:, -1] = 2.0
    q = rounded(q, dtype)
    qd = dev(np.pad(q, ((0, 0),) * 3 + ((0, cache.dim - kr - rd),)), dtype)
    sd, kp = None if sink is None else dev(sink, dtype), pad8(kr)
    out = zeros((B * s_new, H * kp), dtype)
    o = _lib.AttentionOptions(value_dim=kp, sink=ptr(sd))
    _lib.call("rb_attention_general", cuda.ctx, ptr(qd), cache.h, 0, B, s_new, H, scale, ctypes.byref(o), ptr(out), dtype)
    cuda.synchronize()
    cache.close()
    want = np.stack([ref.attention(q[b], c[b][:, None], c[b][:, None, :kr], scale, sink, None, base) for b in range(B)])
    return out.double().cpu().numpy().reshape(B, s_new, H, kp)[..., :kr], want


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,kr,rd", [(4, 64, 16), (6, 72, 32), (12, 128, 64), (16, 200, 24), (5, 45, 6), (32, 512, 64), (20, 256, 0), (3, 512, 100), (70, 64, 32),
                                     (2, 600, 40), (130, 96, 8)])
@pytest.mark.parametrize("base,s_new", [(0, 1), (0, 2), (0, 40), (33, 2), (130, 1), (70, 21)])
def test_attention_over_latents(cuda, dtype, H, kr, rd, base, s_new):
    sink = rounded_sink(np.random.default_rng(H), H, dtype) if kr % 3 else None
    got, want = latent_case(cuda, dtype, H, kr, rd, base, s_new, sink=sink)
    assert rms_err(got, want) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,kr,rd", [(16, 512, 64), (6, 128, 32), (40, 72, 16)])
@pytest.mark.parametrize("T", [1000, 641, 640])
def test_attention_over_many_latents(cuda, dtype, H, kr, rd, T):
    """Single tokens whose keys are shared out over blocks."""
    got, want = latent_case(cuda, dtype, H, kr, rd, T - 1, 1, B=1, sink=rounded_sink(np.random.default_rng(1), H, dtype), seed=3)
    assert rms_err(got, want) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("base,s_new,key", [(64, 1, 0), (64, 1, 63), (64, 1, 64), (127, 1, 64), (128, 1, 127), (0, 129, 128), (0, 129, 0), (0, 129, 64), (60, 9, 63),
                                            (60, 9, 64), (700, 1, 3), (700, 1, 447), (700, 1, 448)])
def test_one_latent_stands_out(cuda, dtype, base, s_new, key):
    got, want = latent_case(cuda, dtype, 5, 72, 16, base, s_new, loud=(key, 3.0), seed=key)
    assert rms_err(got, want) < 2 * TOL[dtype]
    assert np.abs(got[:, -1] - 1.0).max() < 0.05      # (a latent of equal numbers has norm weights of one)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,d,rd,turning,interleaved,kr,e", PRODUCTS[:5] + [(2, 128, 64, 40, False, 600, 200)])
@pytest.mark.parametrize("batch,s_new", [(2, 1), (2, 70), (1, 130)])
def test_heads_of_a_prompt(cuda, dtype, H, d, rd, turning, interleaved, kr, e, batch, s_new):
    """Queries, keys and values where the attention kernels look for them."""
    rng, rows, rot = np.random.default_rng(H + d), batch * s_new, rotation_of(turning, interleaved)
    cache = LatentCache(cuda, latent_dim(dtype, kr, rd), batch, s_new, dtype)
    c = fill_latents(cuda, cache, rng, dtype, batch, s_new, kr, rd)
    cos, sin = tables(cuda, rot, 192) if rot else (None, None)
    widest = max(d + rd, e)
    prompt = Cache(cuda, H, pad8(widest) if dtype == _lib.F32 else next(n for n in (64, 80, 96, 128, 256) if widest <= n), batch, s_new, dtype)
    prompt.set_len(batch, s_new)
    q, k, v = (rounded(rng.standard_normal((batch, s_new, H, n)), dtype) for n in (d + rd, d, e))
    v_col, q_ld = pad8(H * d), pad8(H * (d + rd))
    kv = np.zeros((rows, v_col + pad8(H * e)))
    kv[:, :H * d], kv[:, v_col:v_col + H * e] = k.reshape(rows, -1), v.reshape(rows, -1)
    qs, kvs = dev(padded(q.reshape(rows, -1), q_ld), dtype), dev(kv, dtype)
    out = torch.full((rows, H, prompt.dim), 9.0, dtype=TORCH[dtype], device="cuda")
    _lib.call("rb_latent_heads", cuda.ctx, ptr(qs), q_ld, ptr(kvs), kv.shape[1], v_col, H, d, rd, e, kr, ptr(cos), ptr(sin), turning, int(interleaved), batch,
              s_new, cache.h, 0, prompt.h, ptr(out), dtype)
    cuda.synchronize()
    got = out.double().cpu().numpy().reshape(batch, s_new, H, -1)
    turned = np.stack([ref.rotate(q[b, :, :, d:], rot) for b in range(batch)])
    assert rms_err(got[..., :d], q[..., :d]) == 0 and rms_err(got[..., d:d + rd], turned) < TOL[dtype] and (got[..., d + rd:] == 0).all()
    for b in range(batch):
        for h in range(H):
            kk, vv = prompt.read(b, h, 0, s_new)
            np.testing.assert_array_equal(kk[:, :d + rd], np.concatenate([k[b, :, h], c[b][:, kr:]], -1))
            np.testing.assert_array_equal(vv[:, :e], v[b, :, h])
            assert (kk[:, d + rd:] == 0).all() and (vv[:, e:] == 0).all()
    prompt.close()
    cache.close()
