"""Device buffers of a test of the floating-point op set, in the layouts the ops want (test infrastructure)."""
import numpy as np

import hybrid_oracle as ho


def round8(n):
    return (n + 7) // 8 * 8


class Gpu:
    """Device buffers of one test."""

    def __init__(self, libs):
        self.libs, self.d, self.bufs = libs, libs.cuda(), []
        assert self.d.det_init() == 0

    def put(self, a):
        a = np.ascontiguousarray(a)
        p = self.d.det_malloc(max(a.nbytes, 16))
        self.d.det_memcpy(p, a.ctypes.data, a.nbytes, None)
        self.d.det_sync()
        self.bufs.append(p)
        return p

    def f32(self, a):
        return self.put(np.asarray(a, np.float32))

    def space(self, nbytes):
        p = self.d.det_malloc(max(int(nbytes), 16))
        self.bufs.append(p)
        return p

    def get(self, p, shape, dtype=np.float32):
        out = np.zeros(shape, dtype)
        self.d.det_memcpy(out.ctypes.data, p, out.nbytes, None)
        self.d.det_sync()
        return out

    def act(self, a, dtype, ld=None):
        """Rows in the activation type, padded with zeros to ld; returns the pointer and the values as stored."""
        ld = ld or round8(a.shape[-1])
        full = np.zeros(a.shape[:-1] + (ld,), np.float32)
        full[..., :a.shape[-1]] = a
        if dtype == "f32":
            return self.f32(full), full[..., :a.shape[-1]].astype(float)
        bits = ho.bf16_bits(full)
        return self.put(bits), ho.bf16_values(bits)[..., :a.shape[-1]].astype(float)

    def get_act(self, p, shape, dtype):
        if dtype == "f32":
            return self.get(p, shape).astype(float)
        return ho.bf16_values(self.get(p, shape, np.uint16)).astype(float)

    def linear(self, w):
        """bfloat16 weights; returns the descriptor and the values as stored."""
        n, k = w.shape
        full = np.zeros((n, round8(k)), np.float32)
        full[:, :k] = w
        bits = ho.bf16_bits(full)
        return self.libs.FLinear(self.put(bits), n, k, round8(k)), ho.bf16_values(bits)[:, :k].astype(float)

    def free(self):
        assert self.d.det_last_error() == 0
        for p in self.bufs:
            self.d.det_free(p)


def code(libs, dtype):
    return libs.DET_F32 if dtype == "f32" else libs.DET_BF16


def close(got, want, tol):
    err = np.abs(got - want).max() / max(np.abs(want).max(), 1e-30)
    assert err < tol, err
