"""Helpers of the Malasun GPU tests: the C entry points on torch tensors, and padded layouts."""
import ctypes

import numpy as np
import torch

from rai_b200 import _lib, synth

TORCH = {_lib.BF16: torch.bfloat16, _lib.F32: torch.float32}
DTYPES = [_lib.BF16, _lib.F32]


def ptr(t):
    return None if t is None else ctypes.c_void_p(t.data_ptr())


def pad8(n):
    return (n + 7) // 8 * 8


def rounded(a, dtype):
    """What the GPU will see of `a`: float64 of the value in the model dtype."""
    a = np.asarray(a, dtype=np.float32)
    return (synth.bf16_round(a).reshape(a.shape) if dtype == _lib.BF16 else a).astype(np.float64)


def dev(a, dtype):
    return torch.from_numpy(np.array(a, dtype=np.float32)).to("cuda").to(TORCH[dtype] if dtype in TORCH else dtype).contiguous()


def padded(a, ld):
    """[rows, cols] -> [rows, ld] with zeros."""
    out = np.zeros((a.shape[0], ld), dtype=np.float64)
    out[:, :a.shape[1]] = a
    return out


def rms_err(got, want):
    got = np.asarray(got.float().cpu() if torch.is_tensor(got) else got, dtype=np.float64)
    return float(np.sqrt(((got - want) ** 2).mean()) / (np.sqrt((want ** 2).mean()) + 1e-30))


class Cache:
    """A library KV cache with one layer."""

    def __init__(self, cuda, kv_heads, dim, batch, max_seq, dtype, layers=1):
        self.h = ctypes.c_void_p()
        _lib.call("rb_kv_cache_create", cuda.ctx, layers, kv_heads, dim, batch, max_seq, dtype, ctypes.byref(self.h))
        self.dim, self.dtype = dim, dtype

    def set_len(self, batch, n):
        _lib.call("rb_kv_cache_set_len", self.h, batch, n)

    def read(self, seq, head, t0, n):
        k, v = (torch.empty((n, self.dim), dtype=TORCH[self.dtype]) for _ in range(2))
        _lib.call("rb_kv_cache_read", self.h, 0, seq, head, t0, n, ptr(k), ptr(v))
        return k.double().numpy(), v.double().numpy()

    def close(self):
        _lib.call("rb_kv_cache_destroy", self.h)
