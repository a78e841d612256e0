"""Arrays on the device for the tests of single kernels."""
import numpy as np

import sonuzen_plain as sp
from conftest import load_pkg

pkg = load_pkg()
EPS = 1e-5


def rel(a, b):
    a, b = np.asarray(a, np.float64), np.asarray(b, np.float64)
    return np.linalg.norm(a - b) / max(np.linalg.norm(b), 1e-30)


def pad8(n):
    return (n + 7) // 8 * 8


class Dev:
    """Uploads with automatic release."""

    def __init__(self, gpu):
        self.gpu, self.keep = gpu, []

    def __enter__(self):
        return self

    def __exit__(self, *exc):
        for d in self.keep:
            self.gpu.free(d)

    def up(self, a):
        d = self.gpu.upload(np.ascontiguousarray(a))
        self.keep.append(d)
        return d

    def f32(self, a):
        return self.up(np.asarray(a, np.float32))

    def u32(self, a):
        return self.up(np.asarray(a, np.uint32))

    def bf16(self, a):
        """rows padded with zeros to a multiple of 8 columns"""
        a = np.asarray(a, np.float32)
        out = np.zeros((a.shape[0], pad8(a.shape[1])), np.uint16)
        out[:, :a.shape[1]] = sp.bf16_bits(a)
        return self.up(out)

    def zeros(self, nbytes):
        d = self.gpu.zeros(max(int(nbytes), 16))
        self.keep.append(d)
        return d

    def get(self, d, shape, bf16=False):
        n = int(np.prod(shape))
        if bf16:
            return (self.gpu.download(d, np.uint16, n).astype(np.uint32) << 16).view(np.float32).reshape(shape)
        return self.gpu.download(d, np.float32, n).reshape(shape)

    def call(self, name, *args):
        pkg.check(getattr(self.gpu.lib, name)(self.gpu.handle, *args))
        self.gpu.sync()


def weights(rng, *shape, scale=None):
    return sp.bf16_round(rng.standard_normal(shape).astype(np.float32) * (scale or shape[-1] ** -0.5))
