"""The floating-point op set through the C ABI (include/det_b200.h, Part 3), one mechanism at a time, against the plain functions
of hybrid_oracle.py in float64: both activation types, odd sizes, runs of tokens and single tokens, rings that wrap, rows of
different sequences, keys placed just inside and just outside a window."""
import ctypes as C

import numpy as np
import pytest

import hybrid_oracle as ho
from float_ops import Gpu, close, code, round8

pytestmark = pytest.mark.gpu

TOL = {"f32": 1e-5, "bf16": 1.2e-2}      # of the largest output of a case (fp32 sums over up to 5000 terms)



@pytest.fixture
def gpu(libs):
    g = Gpu(libs)
    yield g
    g.free()


# ------------------------------------------------------------------------------------------------------------------ norm
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("n,m", [(20, 1), (64, 5), (300, 3), (2048, 2), (5000, 7)])
def test_norm_and_rows(dtype, n, m, gpu, libs):
    rng = np.random.default_rng(n + m)
    x, w, rows = rng.standard_normal((9, n)), rng.uniform(0.5, 1.5, n), rng.integers(0, 9, m)
    ld = round8(n) + 8
    op = libs.FNormOp(x=gpu.f32(x), rows=gpu.put(rows.astype(np.int32)), w=gpu.f32(w), eps=0.3, M=m, n=n, dtype=code(libs, dtype),
                      out=gpu.space(m * ld * 4), ld=ld)
    gpu.d.det_f_norm(C.byref(op), None)
    close(gpu.get_act(op.out, (m, ld), dtype)[:, :n], ho.rms_norm(x[rows], 0.3, w), TOL[dtype])


@pytest.mark.parametrize("cut", [[11], [1] * 11, [2, 1, 5, 3], [4, 7]])
def test_token_shift_mixes(cut, gpu, libs):
    """Groups h + (h' - h) mu of a run of tokens, with the previous row carried over every cut."""
    rng = np.random.default_rng(5)
    n, nmix, m = 76, 3, sum(cut)
    x, w, mu = rng.standard_normal((m, n)), rng.uniform(0.5, 1.5, n), rng.uniform(0, 1, (nmix, n))
    h = ho.rms_norm(x, 1e-5, w)
    before = np.vstack([np.zeros(n), h[:-1]])
    want = np.array([h + (before - h) * mu[g] for g in range(nmix)] + [h])
    prev, ld, got, at = gpu.f32(np.zeros(n)), round8(n), [], 0
    for t in cut:
        op = libs.FNormOp(x=gpu.f32(x[at:at + t]), w=gpu.f32(w), eps=1e-5, M=t, n=n, dtype=libs.DET_F32, out=gpu.space(4 * (nmix + 1) * t * ld),
                          ld=ld, group_stride=t * ld, nmix=nmix, mu=gpu.f32(mu), seq=libs.SeqRef(one=libs.SeqSlot(prev=prev)))
        gpu.d.det_f_norm(C.byref(op), None)
        got.append(gpu.get(op.out, (nmix + 1, t, ld))[..., :n])
        at += t
    close(np.concatenate(got, 1), want, TOL["f32"])
    close(gpu.get(prev, n), h[-1], TOL["f32"])


# ------------------------------------------------------------------------------------------------------------------ products
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("flags,m", [(0, m) for m in (1, 2, 3, 4, 5, 31, 33, 127, 130, 300)] + [(f, m) for f in (2, 4) for m in (1, 2, 4, 9, 31)])
def test_products(dtype, flags, m, gpu, libs):
    """Segments with inputs of their own, pair rows, soft cap, accumulation; with and without the GEMV and the split of K."""
    rng = np.random.default_rng(m)
    for n_plain, ff, k in [((7, 130, 5), 37, 76), ((300,), 0, 20), ((64, 64), 520, 1300), ((3,), 8, 9)]:
        groups = len(n_plain)
        n = sum(n_plain) + 2 * ff
        lin, w = gpu.linear(rng.standard_normal((n, k)) / np.sqrt(k))
        ld = round8(k) + 16
        px, x = gpu.act(rng.standard_normal((groups, m + 2, k)), dtype, ld)
        ends = list(np.cumsum(n_plain)) + ([n] if ff else [])
        ins = list(range(groups)) + ([groups - 1] if ff else [])
        y0 = rng.standard_normal((m, sum(n_plain)))
        op = libs.FGemmOp(lin=C.pointer(lin), dtype=code(libs, dtype), x=px, ldx=ld, group_stride=(m + 2) * ld, nseg=len(ends),
                          seg_end=(C.c_int * 8)(*ends), seg_in=(C.c_int * 8)(*ins), glu_from=sum(n_plain), M=m, y=gpu.f32(y0),
                          ldy=sum(n_plain), accumulate=1, h=gpu.space(4 * m * round8(max(ff, 1))), ldh=round8(max(ff, 1)))
        if m % 2:                                        # with and without the tile-major copy of the weights
            ends_c = (C.c_int * 8)(*ends)
            lin.wt = gpu.space(gpu.d.det_f_linear_tile_bytes(k, len(ends), ends_c))
            gpu.d.det_f_linear_tile(C.byref(lin), len(ends), ends_c, lin.wt, None)
        gpu.d.det_debug_set_float(flags)
        try:
            gpu.d.det_f_gemm(C.byref(op), None)
        finally:
            gpu.d.det_debug_set_float(0)
        want, at = np.zeros((m, n)), 0
        for e, g in zip(ends, ins):
            want[:, at:e] = x[g, :m] @ w[at:e].T
            at = e
        close(gpu.get(op.y, y0.shape) - np.float32(y0), want[:, :sum(n_plain)], TOL["f32"])
        if ff:
            g, u = want[:, sum(n_plain)::2], want[:, sum(n_plain) + 1::2]
            close(gpu.get_act(op.h, (m, round8(ff)), dtype)[:, :ff], ho.silu(g) * u, TOL[dtype])


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("m", [1, 3, 9, 140])
def test_product_of_a_norm_with_soft_cap(dtype, m, gpu, libs):
    rng = np.random.default_rng(m)
    for k, n in [(52, 77), (1000, 200), (4096, 24)]:
        lin, w = gpu.linear(rng.standard_normal((n, k)) * 3 / np.sqrt(k))
        x, nw = rng.standard_normal((m, k)) * 4, rng.uniform(0.5, 1.5, k)
        for flags in (0, 1):
            op = libs.FGemmOp(lin=C.pointer(lin), dtype=code(libs, dtype), x=gpu.space(4 * m * round8(k)), ldx=round8(k), nseg=1,
                              seg_end=(C.c_int * 8)(n), glu_from=n, M=m, norm_x=gpu.f32(x), norm_w=gpu.f32(nw), eps=0.1,
                              y=gpu.space(4 * m * n), ldy=n, softcap=2.5)
            gpu.d.det_debug_set_float(flags)
            try:
                gpu.d.det_f_gemm(C.byref(op), None)
            finally:
                gpu.d.det_debug_set_float(0)
            want = 2.5 * np.tanh(ho.rms_norm(x, 0.1, nw) @ w.T / 2.5)
            close(gpu.get(op.y, (m, n)), want, TOL[dtype])


# ------------------------------------------------------------------------------------------------------------------ recurrences
class Recurrence:
    """Random operands of a recurrence and its plain result, token by token."""

    def __init__(self, rng, kind, heads, dk, dv, rank, m):
        self.kind, self.heads, self.dk, self.dv, self.rank, self.m = kind, heads, dk, dv, rank, m
        self.qk, self.vo = heads * dk, heads * dv
        self.y = rng.standard_normal((m, 2 * self.qk + 2 * self.vo + rank)).astype(np.float32)
        # channels that forget at once and channels that hardly forget
        self.bias = rng.uniform(-2, 6, self.qk) if kind == "gla" else rng.uniform(-8, 2, self.qk)
        self.u = None if kind == "gla" else rng.uniform(-1, 2, self.qk)
        self.norm = rng.uniform(0.5, 1.5, self.vo)
        self.w2 = rng.standard_normal((self.qk, rank)) / np.sqrt(rank)
        self.tau, self.scale, self.eps = 3.0, 0.37, 1e-3

    def plain(self, w2, S=None):
        H, dk, dv, out = self.heads, self.dk, self.dv, []
        S = np.zeros((H, dk, dv)) if S is None else S.copy()
        for row in self.y.astype(float):
            q, k, v, g, low = np.split(row, np.cumsum([self.qk, self.qk, self.vo, self.vo]))
            q = q * self.scale
            o = np.zeros((H, dv))
            z = w2 @ (low if self.kind == "gla" else np.tanh(low)) + self.bias
            dec = ho.gla_decay(z, self.tau) if self.kind == "gla" else np.exp(-np.exp(z))
            for h in range(H):
                s = slice(h * dk, (h + 1) * dk)
                if self.kind == "gla":
                    S[h], o[h] = ho.gla_state_step(S[h], q[s], k[s], v[h * dv:(h + 1) * dv], dec[s])
                else:
                    S[h], o[h] = ho.wkv_state_step(S[h], q[s], k[s], v[h * dv:(h + 1) * dv], self.u[s], dec[s])
            out.append(ho.rms_norm(o, self.eps).reshape(-1) * self.norm * ho.silu(g))
        return np.array(out), S

    def op(self, gpu, libs, lin, dtype, rows, **seq):
        y = self.y[rows]
        ld = self.y.shape[1]
        ldo = round8(self.vo) + 8
        op = libs.FRecurOp(heads=self.heads, dk=self.dk, dv=self.dv, rank=self.rank, M=len(y), dtype=code(libs, dtype), y=gpu.f32(y), ldy=ld,
                           q_off=0, k_off=self.qk, v_off=2 * self.qk, gate_off=2 * self.qk + self.vo, low_off=2 * self.qk + 2 * self.vo,
                           q_scale=self.scale, decay=libs.DET_DECAY_SIGMOID if self.kind == "gla" else libs.DET_DECAY_EXP, tau=self.tau,
                           w2=C.pointer(lin), bias=gpu.f32(self.bias), u=None if self.u is None else gpu.f32(self.u),
                           norm=gpu.f32(self.norm), eps=self.eps, out=gpu.space(4 * len(y) * ldo), ldo=ldo,
                           scratch=gpu.space(gpu.d.det_f_recur_scratch_bytes(len(y), self.heads, self.dk, self.dv)), seq=libs.SeqRef(**seq))
        gpu.d.det_f_recur(C.byref(op), None)
        return gpu.get_act(op.out, (len(y), ldo), dtype)[:, :self.vo]


SIZES = [(1, 8, 16, 3), (3, 20, 40, 5), (2, 32, 64, 16), (2, 48, 130, 9), (2, 64, 64, 33), (1, 100, 24, 4), (2, 128, 200, 64), (1, 200, 48, 8),
         (1, 256, 96, 12), (1, 300, 20, 8)]


@pytest.mark.parametrize("kind", ["gla", "wkv"])
@pytest.mark.parametrize("heads,dk,dv,rank", SIZES)
def test_recurrence_sizes(kind, heads, dk, dv, rank, gpu, libs):
    """A run of tokens, the same run one by one, and a mixture, against the plain recurrence; the states must agree too."""
    rng = np.random.default_rng(dk * 7 + dv)
    r = Recurrence(rng, kind, heads, dk, dv, rank, 37)
    lin, w2 = gpu.linear(r.w2)
    want, S = r.plain(w2)
    for cuts in ([37], [1] * 37, [2, 17, 1, 1, 16]):
        state, got, at = gpu.f32(np.zeros((heads, dk, dv))), [], 0
        for t in cuts:
            got.append(r.op(gpu, libs, lin, "f32", slice(at, at + t), one=libs.SeqSlot(s=state)))
            at += t
        close(np.concatenate(got), want, 2e-5)
        close(gpu.get(state, S.shape), S, 1e-5)


@pytest.mark.parametrize("kind", ["gla", "wkv"])
def test_recurrence_activation_type_and_rows(kind, gpu, libs):
    """bfloat16 outputs; a batch whose rows are the next tokens of different sequences."""
    rng = np.random.default_rng(3)
    r = Recurrence(rng, kind, 2, 24, 40, 6, 5)
    lin, w2 = gpu.linear(r.w2)
    close(r.op(gpu, libs, lin, "bf16", slice(0, 5), one=libs.SeqSlot(s=gpu.f32(np.zeros((2, 24, 40))))), r.plain(w2)[0], TOL["bf16"])
    starts = rng.standard_normal((5, 2, 24, 40)).astype(np.float32)
    states = [gpu.f32(s) for s in starts]
    table = gpu.put(np.array([[s, 0, 0] for s in states], np.uint64))
    got = r.op(gpu, libs, lin, "f32", slice(0, 5), table=table, pos=gpu.put(np.zeros(5, np.int32)))
    y = r.y
    for i in range(5):
        r.y = y[i:i + 1]
        want, S = r.plain(w2, starts[i].astype(float))
        close(got[i:i + 1], want, 2e-5)
        close(gpu.get(states[i], S.shape), S, 1e-5)


def test_recurrence_forgets_nothing_over_a_long_run(gpu, libs):
    """A channel whose decay is one to within rounding still holds the first token after 4000 others."""
    rng = np.random.default_rng(8)
    r = Recurrence(rng, "gla", 1, 8, 16, 2, 4000)
    r.bias[:] = 40.0
    r.y[1:, r.qk:2 * r.qk] = 0.0                    # only the first token writes
    lin, w2 = gpu.linear(r.w2 * 0)
    state = gpu.f32(np.zeros((1, 8, 16)))
    got = r.op(gpu, libs, lin, "f32", slice(0, 4000), one=libs.SeqSlot(s=state))
    close(got[-1:], r.plain(w2)[0][-1:], 1e-4)


# ------------------------------------------------------------------------------------------------------------------ latent attention
class Latent:
    def __init__(self, rng, n, heads, dim, rot, vdim, q_rank, kv_rank, window, base=300.0):
        self.n, self.heads, self.dim, self.rot, self.vdim, self.q_rank, self.kv_rank, self.window = n, heads, dim, rot, vdim, q_rank, kv_rank, window
        self.base, self.scale, self.eps = base, 0.3, 1e-4
        self.hd = dim + rot
        self.y = rng.standard_normal((n, q_rank + kv_rank + rot + heads * vdim)).astype(np.float32)
        self.dqn, self.dkvn = rng.uniform(0.5, 1.5, q_rank), rng.uniform(0.5, 1.5, kv_rank)
        self.q = rng.standard_normal((n, heads * self.hd)).astype(np.float32)
        self.wkv = rng.standard_normal((heads * (dim + vdim), kv_rank)) / np.sqrt(kv_rank)
        self.sink = rng.uniform(-1, 2, heads)

    def plain(self, w, window=None):
        """(normalised query latents, gated outputs); the keys and values of the cache are multiplied out per head."""
        window = self.window if window is None else window
        R, H, d, rd, dv = self.kv_rank, self.heads, self.dim, self.rot, self.vdim
        y, q = self.y.astype(float), self.q.astype(float).reshape(self.n, H, self.hd)
        c = ho.rms_norm(y[:, self.q_rank:self.q_rank + R], self.eps, self.dkvn)
        kr = np.array([ho.rotate_pairs(y[p, self.q_rank + R:self.q_rank + R + rd], p, self.base, rd) for p in range(self.n)])
        K, V = c @ w[:H * d].T, c @ w[H * d:].T
        out = np.zeros((self.n, H * dv))
        for i in range(self.n):
            lo = max(0, i - window + 1) if window > 0 else 0
            for h in range(H):
                s = K[lo:i + 1, h * d:(h + 1) * d] @ q[i, h, :d] + kr[lo:i + 1] @ ho.rotate_pairs(q[i, h, d:], i, self.base, rd)
                out[i, h * dv:(h + 1) * dv] = ho.softmax_with_sink(s * self.scale, self.sink[h]) @ V[lo:i + 1, h * dv:(h + 1) * dv]
        return ho.rms_norm(y[:, :self.q_rank], self.eps, self.dqn), out * ho.sigmoid(y[:, self.q_rank + R + rd:])

    def setup(self, gpu, libs, dtype, cap):
        self.lin, w = gpu.linear(self.wkv)
        self.ld = gpu.d.det_f_latent_ld(self.kv_rank, self.rot)
        a = np.arange(self.n + 1)[:, None] * self.base ** (-2.0 * np.arange(self.rot // 2) / max(self.rot, 1))
        self.cos, self.sin = gpu.f32(np.cos(a)), gpu.f32(np.sin(a))
        self.cap, self.dtype = cap, dtype
        self.consts = [gpu.f32(self.dqn), gpu.f32(self.dkvn), gpu.f32(self.sink)]
        return w

    def cache(self, gpu):
        return gpu.space(self.cap * self.ld * 4)

    def op(self, gpu, libs, rows, max_pos, **seq):
        R, H = self.kv_rank, self.heads
        idx = np.arange(self.n)[rows] if isinstance(rows, slice) else np.asarray(rows)
        m, ldo, ldcq = len(idx), round8(H * self.vdim) + 8, round8(self.q_rank)
        scratch = gpu.d.det_f_latent_scratch_bytes(m, H, self.dim, self.rot, self.vdim, R, self.window, self.cap, max_pos, code(libs, self.dtype))
        op = libs.FLatentOp(heads=H, dim=self.dim, rot_dim=self.rot, rot_dims=self.rot, vdim=self.vdim, q_rank=self.q_rank, kv_rank=R,
                            window=self.window, scale=self.scale, cap=self.cap, M=m, dtype=code(libs, self.dtype), y=gpu.f32(self.y[idx]),
                            ldy=self.y.shape[1], dq_off=0, dkv_off=self.q_rank, gate_off=self.q_rank + R + self.rot, dq_norm=self.consts[0],
                            dkv_norm=self.consts[1], eps=self.eps, rope_cos=self.cos, rope_sin=self.sin, cq=gpu.space(4 * m * ldcq), ldcq=ldcq,
                            q=gpu.f32(self.q[idx]), ldq=H * self.hd, wkv=C.pointer(self.lin), sink=self.consts[2],
                            out=gpu.space(4 * m * ldo), ldo=ldo, max_pos=max_pos, scratch=gpu.space(scratch), seq=libs.SeqRef(**seq))
        gpu.d.det_f_latent_prep(C.byref(op), None)
        gpu.d.det_f_latent_attn(C.byref(op), None)
        return gpu.get_act(op.cq, (m, ldcq), self.dtype)[:, :self.q_rank], gpu.get_act(op.out, (m, ldo), self.dtype)[:, :H * self.vdim]

    def run(self, gpu, libs, cuts, cache):
        got, at = [], 0
        for t in cuts:
            got.append(self.op(gpu, libs, slice(at, at + t), at + t - 1, one=libs.SeqSlot(cache=cache), pos0=at))
            at += t
        return [np.concatenate(x) for x in zip(*got)]


SHAPES = [dict(heads=1, dim=8, rot=2, vdim=8, q_rank=9, kv_rank=10, window=1), dict(heads=3, dim=20, rot=6, vdim=12, q_rank=30, kv_rank=50, window=7),
          dict(heads=6, dim=32, rot=8, vdim=40, q_rank=40, kv_rank=24, window=64), dict(heads=9, dim=16, rot=16, vdim=72, q_rank=64, kv_rank=130, window=33),
          dict(heads=2, dim=40, rot=24, vdim=136, q_rank=16, kv_rank=320, window=129), dict(heads=4, dim=64, rot=8, vdim=200, q_rank=24, kv_rank=64, window=0)]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("shape", range(len(SHAPES)))
def test_latent_attention(dtype, shape, gpu, libs):
    """Whole prompts, single tokens and portions over a cache that is a ring just as large as the largest portion needs."""
    s = SHAPES[shape]
    n = 300
    a = Latent(np.random.default_rng(shape), n, **s)
    for cuts in ([n], [140] + [1] * 20 + [2, 33, 64, 41], [2, 3, 37] * 6 + [1] * 48):
        assert sum(cuts) == n
        cap = min(n, s["window"] - 1 + max(cuts)) if s["window"] else n
        w = a.setup(gpu, libs, dtype, cap)
        want_cq, want = a.plain(w)
        cq, out = a.run(gpu, libs, cuts, a.cache(gpu))
        close(cq, want_cq, TOL[dtype])
        close(out, want, 2e-5 if dtype == "f32" else 3e-2)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("window", [1, 2, 16, 17, 63, 64, 65, 128, 200])
def test_keys_at_the_window_edge(dtype, window, gpu, libs):
    """One key per query dominates every other by far.  Placed on the last position that the window keeps it must decide the
    output, one position further back it must not be there at all; the same for a key next to the query."""
    n = 330
    a = Latent(np.random.default_rng(window), n, heads=2, dim=16, rot=8, vdim=16, q_rank=8, kv_rank=16, window=window)
    a.q *= 0.1
    a.sink[:] = -5.0
    R = a.kv_rank
    # all latents point along axis 0; key `j` of a few positions along axis 1, which the chosen queries look for
    a.y[:, 8:8 + R] = 0.01 * a.y[:, 8:8 + R]
    a.y[:, 8] = 1.0
    a.wkv[:2 * 16] *= 0.05
    a.wkv[0, 1] = a.wkv[16, 1] = 4.0
    for j in (0, 5, 60, 63, 64, 127, 128, 129):
        a.y[j, 8:8 + R] = 0.0
        a.y[j, 9] = 1.0
        for i in (j + window - 1, j + window):
            if i < n:
                a.q[i].reshape(2, -1)[:, 0] = 12.0
    w = a.setup(gpu, libs, dtype, window - 1 + 250)
    want = a.plain(w)[1]
    assert np.abs(a.plain(w, window + 1)[1] - want).max() > 0.3 * np.abs(want).max()
    if window > 1:
        assert np.abs(a.plain(w, window - 1)[1] - want).max() > 0.3 * np.abs(want).max()
    for cuts in ([250] + [1] * 80, [130, 2, 35, 1, 1, 80] + [1] * 81, [40] + [3] * 30 + [200]):
        close(a.run(gpu, libs, cuts, a.cache(gpu))[1], want, 2e-5 if dtype == "f32" else 3e-2)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_latent_rows_of_different_sequences(dtype, gpu, libs):
    """A step over sequences of unequal lengths equals each alone; a cache used by an ended sequence serves another."""
    a = Latent(np.random.default_rng(4), 90, heads=5, dim=24, rot=8, vdim=16, q_rank=16, kv_rank=40, window=21)
    w = a.setup(gpu, libs, dtype, 21 - 1 + 60)
    want = a.plain(w)[1]
    lengths = [1, 20, 21, 22, 59, 89]
    caches = [a.cache(gpu) for _ in lengths]
    for cache in caches:                              # an earlier conversation fills every row of the ring
        a.run(gpu, libs, [60, 30], cache)
    for cache, n in zip(caches, lengths):
        a.run(gpu, libs, [min(n, 60)] + [1] * (n - min(n, 60)), cache)
    table = gpu.put(np.array([[0, 0, c] for c in caches], np.uint64))
    got = a.op(gpu, libs, lengths, 89, table=table, pos=gpu.put(np.array(lengths, np.int32)))[1]
    close(got, want[lengths], 2e-5 if dtype == "f32" else 3e-2)
