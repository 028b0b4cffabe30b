"""The ops of the serial layers through the C ABI, one mechanism at a time, against the plain functions of dopipel_oracle.py in
float64: both activation types, odd sizes, cuts of a run, rows of different sequences, single keys that stand out."""
import ctypes as C

import numpy as np
import pytest

import dopipel_oracle as do
import hybrid_oracle as ho
from float_ops import Gpu, close, code, round8

pytestmark = pytest.mark.gpu

TOL = {"f32": 1e-5, "bf16": 1.2e-2}


@pytest.fixture
def gpu(libs):
    g = Gpu(libs)
    yield g
    g.free()


def slots(gpu, libs, entries):
    """Device table of sequence slots."""
    return gpu.put(np.frombuffer(b"".join(bytes(libs.SeqSlot(**e)) for e in entries), np.uint8))


# ------------------------------------------------------------------------------------------------------------------ seams
def seam_reference(x, y, yn, ys, w, conv, eps, past):
    out = []
    for t in range(len(x)):
        if y is not None:
            x[t] = x[t] + ho.rms_norm(y[t], eps, yn) * (1.0 if ys is None else ys)
        h = x[t] if w is None else ho.rms_norm(x[t], eps, w)
        if conv is not None:
            add, past = do.causal_conv(conv, h, past)
            h = h + add
        out.append(h)
    return np.array(out), past


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("n", [20, 77, 1024, 5120])
@pytest.mark.parametrize("m", [1, 6, 160])
def test_seam_without_convolution(n, m, dtype, gpu, libs):
    """Result norm, layer scale, residual add and the next norm; without parts of them."""
    rng = np.random.default_rng(n + m)
    ld, ldy = round8(n) + 8, n + 4
    yn, ys, w = rng.uniform(0.5, 1.5, (3, n))
    for use_y, use_s, use_w, use_out in [(1, 1, 1, 1), (1, 0, 0, 1), (0, 0, 1, 1), (0, 0, 0, 1), (1, 1, 1, 0)]:
        x, y = rng.standard_normal((m, n)), 3 * rng.standard_normal((m, ldy))
        px = gpu.f32(x)
        op = libs.FSeamOp(x=px, M=m, n=n, eps=0.01, y=gpu.f32(y) if use_y else None, ldy=ldy, y_norm=gpu.f32(yn),
                          y_scale=gpu.f32(ys) if use_s else None, w=gpu.f32(w) if use_w else None, dtype=code(libs, dtype),
                          out=gpu.space(4 * m * ld) if use_out else None, ld=ld)
        gpu.d.det_f_seam(C.byref(op), None)
        want, _ = seam_reference(x, y[:, :n] if use_y else None, yn, ys if use_s else None, w if use_w else None, None, 0.01, None)
        close(gpu.get(px, (m, n)), x, TOL["f32"])
        if use_out:
            close(gpu.get_act(op.out, (m, ld), dtype)[:, :n], want, TOL[dtype])


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 9, 16])
@pytest.mark.parametrize("n", [24, 53, 1100])
def test_seam_with_convolution_over_cuts(n, taps, gpu, libs):
    """One sequence in portions down to one token: the latest rows carry over every cut, whatever its size beside the taps."""
    rng = np.random.default_rng(n + taps)
    w, yn = rng.uniform(0.5, 1.5, (2, n))
    conv = rng.standard_normal((n, taps))
    ld = round8(n)
    for cut in ([75], [1] * 20, [2, 1, 3, 2, 2, 17, 16, 2], [33, 15, 16, 1, 7], [4, 40, 2]):
        m = sum(cut)
        x, y = rng.standard_normal((m, n)), rng.standard_normal((m, n))
        x0 = x.copy()
        want, past = seam_reference(x, y, yn, None, w, conv, 1e-5, np.zeros((taps - 1, n)))
        prev, rstd, got, at = gpu.f32(np.zeros((max(1, taps - 1), n))), gpu.space(4 * m), [], 0
        for t in cut:
            op = libs.FSeamOp(x=gpu.f32(x0[at:at + t]), M=t, n=n, eps=1e-5, y=gpu.f32(y[at:at + t]), ldy=n, y_norm=gpu.f32(yn), w=gpu.f32(w),
                              conv=gpu.f32(conv.T), taps=taps, rstd=rstd, dtype=libs.DET_F32, out=gpu.space(4 * t * ld), ld=ld,
                              seq=libs.SeqRef(one=libs.SeqSlot(prev=prev)))
            gpu.d.det_f_seam(C.byref(op), None)
            got.append(gpu.get(op.out, (t, ld))[:, :n])
            close(gpu.get(op.x, (t, n)), x[at:at + t], TOL["f32"])
            at += t
        close(np.concatenate(got), want, TOL["f32"])
        if taps > 1:
            close(gpu.get(prev, (taps - 1, n)), past, TOL["f32"])


@pytest.mark.parametrize("rows", [1, 5, 200])
def test_seam_rows_of_different_sequences(rows, gpu, libs):
    rng = np.random.default_rng(rows)
    n, taps = 72, 4
    w, conv, prev = rng.uniform(0.5, 1.5, n), rng.standard_normal((n, taps)), rng.standard_normal((rows, taps - 1, n))
    x = rng.standard_normal((rows, n))
    p = [gpu.f32(prev[r]) for r in range(rows)]
    op = libs.FSeamOp(x=gpu.f32(x), M=rows, n=n, eps=1e-5, w=gpu.f32(w), conv=gpu.f32(conv.T), taps=taps, dtype=libs.DET_F32,
                      out=gpu.space(4 * rows * n), ld=n, seq=libs.SeqRef(table=slots(gpu, libs, [{"prev": q} for q in p])))
    gpu.d.det_f_seam(C.byref(op), None)
    got = gpu.get(op.out, (rows, n))
    for r in range(rows):
        want, past = seam_reference(x[r:r + 1].copy(), None, None, None, w, conv, 1e-5, prev[r])
        close(got[r:r + 1], want, TOL["f32"])
        close(gpu.get(p[r], (taps - 1, n)), past, TOL["f32"])


# ------------------------------------------------------------------------------------------------------------------ products
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("flags,m", [(0, 1), (0, 2), (0, 4), (0, 7), (0, 40), (0, 150), (2, 3), (4, 9)])
def test_products_with_biases_and_activations(flags, m, dtype, gpu, libs):
    rng = np.random.default_rng(m)
    for act, plain, ff, k in [(libs.DET_FF_REGLU, 0, 60, 76), (libs.DET_FF_REGLU, 9, 36, 200), (libs.DET_FF_RELU2, 21, 35, 136),
                              (libs.DET_FF_RELU2, 0, 130, 52), (libs.DET_FF_SWIGLU, 150, 0, 1300)]:
        rows = ff if act == libs.DET_FF_RELU2 else 2 * ff
        lin, w = gpu.linear(rng.standard_normal((plain + rows, k)) / np.sqrt(k))
        ld, ldh = round8(k), round8(max(1, ff))
        px, x = gpu.act(rng.standard_normal((m, k)), dtype)
        bias = rng.standard_normal(max(1, plain))
        ends = ([plain] if plain else []) + ([plain + rows] if rows else [])
        op = libs.FGemmOp(lin=C.pointer(lin), dtype=code(libs, dtype), x=px, ldx=ld, nseg=len(ends), seg_end=(C.c_int * 8)(*ends), glu_from=plain,
                          M=m, y=gpu.space(4 * m * max(1, plain)), ldy=plain, h=gpu.space(4 * m * ldh), ldh=ldh, bias=gpu.f32(bias), act=act)
        gpu.d.det_debug_set_float(flags)
        try:
            gpu.d.det_f_gemm(C.byref(op), None)
        finally:
            gpu.d.det_debug_set_float(0)
        want = x @ w.T
        if plain:
            close(gpu.get(op.y, (m, plain)), want[:, :plain] + np.float32(bias), TOL["f32"])
        if ff:
            v = want[:, plain:]
            h = np.square(np.maximum(v, 0)) if act == libs.DET_FF_RELU2 else np.maximum(v[:, 0::2], 0) * v[:, 1::2]
            close(gpu.get_act(op.h, (m, ldh), dtype)[:, :ff], h, TOL[dtype])


# ------------------------------------------------------------------------------------------------------------------ attention
class Attention:
    """One sequence of an attention case: rows y as the projections leave them and the cache they go through."""

    def __init__(self, gpu, libs, dtype, heads, kv_heads, dim, vdim, rot, cap, gated=True, vrot=True, seed=0):
        self.gpu, self.libs, self.dtype = gpu, libs, dtype
        self.H, self.G, self.d, self.dv, self.rot, self.cap = heads, kv_heads, dim, vdim, rot, cap
        self.gated, self.vrot, self.base, self.scale = gated, vrot, 300.0, 0.7 / np.sqrt(dim)
        self.n = heads * dim + kv_heads * (dim + vdim) + (heads if gated else 0)
        self.rng = np.random.default_rng(seed)
        self.cache = gpu.space(4 * cap * gpu.d.det_f_attn_ld(kv_heads, dim, vdim))
        pos = np.arange(cap)[:, None]

        def table(dims):
            a = pos * np.power(self.base, -2.0 * np.arange(dims // 2) / max(dims, 1))[None]
            return gpu.f32(np.append(np.cos(a), 0)), gpu.f32(np.append(np.sin(a), 0))
        self.kt, self.vt = table(rot), table(vdim)
        self.scratch = gpu.space(gpu.d.det_f_attn_scratch_bytes(vdim))

    def rows(self, n, aim):
        """Projections of n tokens.  aim[t]: the earlier position on which every head of token t puts its weight."""
        y = self.rng.standard_normal((n, self.n))
        k = y[:, self.H * self.d:self.H * self.d + self.G * self.d].reshape(n, self.G, self.d)
        for t, j in aim.items():
            for h in range(self.H):
                kj = ho.rotate_pairs(k[j, h * self.G // self.H], j, self.base, self.rot)
                q = 25.0 / (self.scale * kj @ kj) * kj
                y[t, h * self.d:(h + 1) * self.d] = ho.rotate_pairs(q, -t, self.base, self.rot)
        return y

    def reference(self, y):
        H, G, d, dv = self.H, self.G, self.d, self.dv
        K, V, out = [], [], []
        for t, r in enumerate(y):
            q, k, v = np.split(r[:H * d + G * (d + dv)], [H * d, H * d + G * d])
            q, k = (ho.rotate_pairs(a.reshape(-1, d), t, self.base, self.rot) for a in (q, k))
            turn = self.base if self.vrot else None
            v = v.reshape(G, dv)
            K.append(k)
            V.append(ho.rotate_pairs(v, t, turn, dv) if turn else v)
            o = np.zeros((H, dv))
            for h in range(H):
                g = h * G // H
                p = do.attention_weights(q[h], np.array(K)[:, g], self.scale)
                o[h] = p @ np.array(V)[:, g]
                if turn:
                    o[h] = ho.rotate_pairs(o[h], -t, turn, dv)
                if self.gated:
                    o[h] *= ho.sigmoid(r[-H + h])
            out.append(o.reshape(-1))
        return np.array(out)

    def op(self, y, seq, max_pos):
        m, H, G, d, dv = len(y), self.H, self.G, self.d, self.dv
        ldo = round8(H * dv)
        return self.libs.FAttnOp(heads=H, kv_heads=G, dim=d, vdim=dv, rot_dims=self.rot, scale=self.scale, cap=self.cap, M=m,
                                 dtype=code(self.libs, self.dtype), y=self.gpu.f32(y), ldy=self.n, q_off=0, k_off=H * d, v_off=(H + G) * d,
                                 gate_off=(H + G) * d + G * dv if self.gated else -1, rope_cos=self.kt[0], rope_sin=self.kt[1],
                                 vrope_cos=self.vt[0] if self.vrot else None, vrope_sin=self.vt[1] if self.vrot else None,
                                 q=self.gpu.space(4 * m * self.gpu.d.det_f_attn_q_ld(H, d)), out=self.gpu.space(4 * m * ldo), ldo=ldo,
                                 max_pos=max_pos, scratch=self.scratch, seq=seq)

    def run(self, y, pos0, pos=None):
        seq = self.libs.SeqRef(one=self.libs.SeqSlot(cache=self.cache), pos0=0 if pos else pos0, pos=pos)
        op = self.op(y, seq, self.cap - 1 if pos else pos0 + len(y) - 1)
        self.gpu.d.det_f_attn_prep(C.byref(op), None)
        self.gpu.d.det_f_attn(C.byref(op), None)
        return self.gpu.get_act(op.out, (len(y), op.ldo), self.dtype)[:, :self.H * self.dv]


SHAPES = [(6, 2, 40, 24, 24), (1, 1, 16, 8, 16), (5, 5, 20, 12, 10), (3, 1, 11, 30, 0), (20, 1, 64, 64, 32), (8, 2, 128, 128, 128),
          (4, 4, 72, 136, 8), (2, 1, 256, 200, 64), (2, 2, 24, 256, 24), (2, 1, 320, 272, 100)]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("shape", SHAPES, ids=str)
def test_attention_over_cuts(shape, dtype, gpu, libs):
    """Keys far away, at the edges of the kernels' tiles and splits, and the first token, asked for in prompts and in decoding."""
    n = 300
    aim = {t: j for t, j in [(63, 0), (64, 0), (65, 64), (127, 64), (128, 63), (130, 1), (191, 127), (192, 128), (200, 0), (255, 254),
                             (256, 65), (257, 0), (260, 3), (270, 270), (280, 16), (281, 15), (290, 191), (298, 47), (299, 0)]}
    a = Attention(gpu, libs, dtype, *shape, cap=n + 3, seed=n)
    y = a.rows(n, aim)
    want = a.reference(np.float32(y).astype(float))
    for cut in ([n], [40] + [1] * 30 + [130, 2, 3, 31, 33] + [1] * 31, [257, 2, 41]):
        at = 0
        got = []
        for t in cut:
            got.append(a.run(y[at:at + t], at))
            at += t
        got = np.concatenate(got)
        close(got, want, 3 * TOL[dtype])
        planted = sorted(aim)
        close(got[planted], want[planted], 3 * TOL[dtype])


@pytest.mark.parametrize("gated,vrot", [(False, True), (True, False), (False, False)])
def test_attention_without_gate_or_rotated_values(gated, vrot, gpu, libs):
    for dtype in TOL:
        a = Attention(gpu, libs, dtype, 4, 2, 24, 16, 16, cap=90, gated=gated, vrot=vrot)
        y = a.rows(90, {80: 2, 89: 40})
        want = a.reference(np.float32(y).astype(float))
        close(np.concatenate([a.run(y[:50], 0), a.run(y[50:85], 50)] + [a.run(y[i:i + 1], i) for i in range(85, 90)]), want, 3 * TOL[dtype])


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_attention_rows_of_different_sequences(dtype, gpu, libs):
    """A batch of unequal positions, each against its own cache, and the position word of a captured step."""
    lengths = [1, 2, 64, 65, 127, 200, 31]
    seqs, rows, want = [], [], []
    for i, n in enumerate(lengths):
        a = Attention(gpu, libs, dtype, 6, 3, 40, 32, 40, cap=210, seed=i)
        y = a.rows(n, {n - 1: 0})
        want.append(a.reference(np.float32(y).astype(float))[-1])
        if n > 1:
            a.run(y[:-1], 0)
        seqs.append(a)
        rows.append(y[-1])
    a = seqs[0]
    seq = libs.SeqRef(table=slots(gpu, libs, [{"cache": s.cache} for s in seqs]), pos=gpu.put(np.array(lengths, np.int32) - 1))
    op = a.op(np.array(rows), seq, max(lengths) - 1)
    gpu.d.det_f_attn_prep(C.byref(op), None)
    gpu.d.det_f_attn(C.byref(op), None)
    got = gpu.get_act(op.out, (len(rows), op.ldo), dtype)[:, :a.H * a.dv]
    close(got, np.array(want), 3 * TOL[dtype])
    for s, n, r, w in zip(seqs, lengths, rows, want):
        close(s.run(r[None], n - 1, pos=gpu.put(np.array([n - 1], np.int32))), w[None], 3 * TOL[dtype])


# ------------------------------------------------------------------------------------------------------------------ recurrence
@pytest.mark.parametrize("n,m", [(5, 70), (40, 300), (300, 41), (33, 600)])
def test_minimal_gated_recurrence(n, m, gpu, libs):
    rng = np.random.default_rng(n)
    y = rng.standard_normal((m, 3 * n + 2)) * 2
    y[:, :n] -= 3.0                                         # slow channels: the state reaches far back
    S, want = np.zeros(n), []
    yf = np.float32(y).astype(float)
    for r in yf:
        z = ho.sigmoid(r[:n])
        S = (1 - z) * S + z * do.mingru_candidate(r[n:2 * n])
        want.append(S * ho.silu(r[2 * n:3 * n]))
    for dtype in TOL:
        for cut in ([m], [1] * 20 + [m - 20], [2, 3, 8, 9, 7, m - 29]):
            state, got, at = gpu.f32(np.zeros(n)), [], 0
            for t in cut:
                op = libs.FMinGruOp(n=n, M=t, dtype=code(libs, dtype), y=gpu.f32(y[at:at + t]), ldy=3 * n + 2, z_off=0, x_off=n, gate_off=2 * n,
                                    out=gpu.space(4 * t * round8(n)), ldo=round8(n), seq=libs.SeqRef(one=libs.SeqSlot(s=state)))
                gpu.d.det_f_mingru(C.byref(op), None)
                got.append(gpu.get_act(op.out, (t, round8(n)), dtype)[:, :n])
                at += t
            close(np.concatenate(got), np.array(want), TOL[dtype])
            close(gpu.get(state, n), S, TOL["f32"])
    states = [gpu.f32(rng.standard_normal(n)) for _ in range(9)]
    before = [gpu.get(s, n).astype(float) for s in states]
    op = libs.FMinGruOp(n=n, M=9, dtype=libs.DET_F32, y=gpu.f32(y[:9]), ldy=3 * n + 2, z_off=0, x_off=n, gate_off=2 * n,
                        out=gpu.space(4 * 9 * round8(n)), ldo=round8(n), seq=libs.SeqRef(table=slots(gpu, libs, [{"s": s} for s in states])))
    gpu.d.det_f_mingru(C.byref(op), None)
    for r in range(9):
        z = ho.sigmoid(yf[r, :n])
        close(gpu.get(states[r], n), (1 - z) * before[r] + z * do.mingru_candidate(yf[r, n:2 * n]), TOL["f32"])


# ------------------------------------------------------------------------------------------------------------------ mixture
MIXTURES = [dict(experts=10, identity=3, top=3, ff=40, n=96, shared=56), dict(experts=3, identity=0, top=1, ff=9, n=52, shared=0),
            dict(experts=1, identity=4, top=2, ff=24, n=64, shared=8), dict(experts=60, identity=10, top=8, ff=72, n=136, shared=20),
            dict(experts=300, identity=20, top=40, ff=16, n=64, shared=0), dict(experts=4, identity=1, top=5, ff=200, n=300, shared=33)]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("case", MIXTURES, ids=lambda c: "-".join(str(v) for v in c.values()))
def test_mixture_of_experts(case, dtype, gpu, libs):
    """Few rows (a pair streams its expert) and more (rows sorted by expert), with and without the tile-major copies; all rows on
    one expert; only identity experts."""
    E, I, top, ff, n, sf = case.values()
    rng = np.random.default_rng(E)
    up, wu = gpu.linear(rng.standard_normal((E * ff, n)) / np.sqrt(n))
    down, wd = gpu.linear(rng.standard_normal((E * n, ff)) / np.sqrt(ff))
    if sf:
        sd, ws = gpu.linear(rng.standard_normal((n, sf)) / np.sqrt(sf))
    corr = rng.uniform(-0.05, 0.05, E + I)
    counts = gpu.put(np.zeros(libs.DET_MAX_ROUTER + 1, np.uint32))
    ld, ldz = round8(n), E + I + 3
    for tiled, m in [(0, 1), (0, 3), (0, 4), (0, 5), (1, 30), (0, 70), (1, 260)]:
        if tiled:
            for lin in (up, down):
                lin.wt = gpu.space(gpu.d.det_f_linear_tile_groups_bytes(lin.K, E, lin.N // E))
                gpu.d.det_f_linear_tile_groups(C.byref(lin), E, lin.wt, None)
        px, x = gpu.act(rng.standard_normal((m, n)), dtype)
        z = rng.standard_normal((m, ldz)) * 2
        if m == 70:
            z[:, 0] += 30.0
        if m == 5 and I >= top:
            z[:, E:E + I] += 40.0
        if sf:
            ph, hs = gpu.act(np.square(np.maximum(rng.standard_normal((m, sf)), 0)), dtype)
        op = libs.FMoeOp(experts=E, identity=I, top=top, ff=ff, n=n, M=m, dtype=code(libs, dtype), z=gpu.f32(z), ldz=ldz,
                         correction=gpu.f32(corr), x=px, ldx=ld, up=C.pointer(up), down=C.pointer(down), shared=C.pointer(sd) if sf else None,
                         hs=ph if sf else None, ldhs=round8(max(sf, 1)), shared_gate=E + I if sf else -1, out=gpu.space(4 * m * n), ldo=n,
                         counts=counts, scratch=gpu.space(gpu.d.det_f_moe_scratch_bytes(m, E, top, ff, n, code(libs, dtype))))
        gpu.d.det_f_moe(C.byref(op), None)
        want = np.zeros((m, n))
        zf = np.float32(z).astype(float)
        for r in range(m):
            for e, p in zip(*do.route(zf[r, :E + I], np.float32(corr), top)):
                want[r] += p * (x[r] if e >= E else do.expert_ff(wu[e * ff:(e + 1) * ff], wd[e * n:(e + 1) * n], x[r]))
            if sf:
                want[r] += ho.sigmoid(zf[r, E + I]) * (ws @ hs[r])
        close(gpu.get(op.out, (m, n)), want, TOL[dtype])
        assert not gpu.get(counts, libs.DET_MAX_ROUTER + 1, np.uint32).any()
