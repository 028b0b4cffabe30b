// Causal attention of a run of tokens on bfloat16 MMAs, shared by the attention kernels: 64 query rows of one head against
// 64-key tiles, online softmax in 32-bit, keys and values by asynchronous copies one tile ahead.  What a query, a key row and an
// output row are is the source's business (a small struct per kind of attention):
//   unsigned query(row, pos, e)     elements e, e + 1 of the scaled query (log-2 units), zeros past its end
//   int pieces(), FlashPiece piece(v)     the 16-byte pieces of a key / value row and where they go
//   float inverse(m, l)             factor on the summed values, from the row's maximum and sum
//   void store(row, pos, v, o0, o1) output elements v, v + 1
#pragma once
#include "fops.cuh"

namespace detb {

constexpr int FL_ROWS = 64, FL_KEYS = 64, FL_WARPS = 4;

struct FlashShape {
    int hd;          // query / key dimensions
    int window;      // keys a row sees, itself included; 0: all
    int cap;         // rows of the cache ring
    int M;           // query rows of the call
};
struct FlashPiece {
    const bf16* p;   // of cache slot 0
    int step;        // elements to the next slot
    int vec;         // 16-byte piece of the staged row
    bool value;
};

__device__ __forceinline__ int first_key(int pos, int window) { return window > 0 ? max(0, pos - window + 1) : 0; }

__device__ __forceinline__ void ldsm4(unsigned addr, unsigned (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4_t(unsigned addr, unsigned (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma16816(float (&d)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp_async16(unsigned dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// 2^x by the special function unit (relative error about 2^-22; 2^-inf = 0).
__device__ __forceinline__ float exp2_fast(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

inline size_t flash_smem(int hd, int dv) {
    const int ldk = ((hd + 15) & ~15) + 8;
    return ((size_t)(FL_ROWS + 2 * FL_KEYS) * ldk + 2 * (size_t)FL_KEYS * (dv + 8)) * 2;
}

// Scores of a 16-row warp tile against NB * 8 keys, then the rows' running maximum, sum and weights.  Rows past M and masked
// scores take part as -inf.
struct FlashRows {
    float m[2], l[2];
};
template <int NB, int NO>
__device__ __forceinline__ void flash_softmax(FlashRows& r, float (&s)[NB][4], float (&o)[NO][4], unsigned (&pf)[NB / 2][4]) {
    float mx[2] = {r.m[0], r.m[1]};
#pragma unroll
    for (int n = 0; n < NB; n++) {
        mx[0] = fmaxf(mx[0], fmaxf(s[n][0], s[n][1]));
        mx[1] = fmaxf(mx[1], fmaxf(s[n][2], s[n][3]));
    }
#pragma unroll
    for (int i = 0; i < 2; i++) {
        mx[i] = fmaxf(mx[i], __shfl_xor_sync(FULL, mx[i], 1));
        mx[i] = fmaxf(mx[i], __shfl_xor_sync(FULL, mx[i], 2));
    }
    float f[2], base[2];
#pragma unroll
    for (int i = 0; i < 2; i++) {
        base[i] = mx[i] == -INFINITY ? 0.0f : mx[i];       // no key seen yet: every weight below is exp2(-inf) = 0
        f[i] = exp2_fast(r.m[i] - base[i]);
        r.m[i] = mx[i];
        r.l[i] *= f[i];
    }
    if (__any_sync(FULL, f[0] != 1.0f || f[1] != 1.0f)) {
#pragma unroll
        for (int i = 0; i < NO; i++) {
            o[i][0] *= f[0];
            o[i][1] *= f[0];
            o[i][2] *= f[1];
            o[i][3] *= f[1];
        }
    }
#pragma unroll
    for (int n = 0; n < NB; n++) {
        const float e0 = exp2_fast(s[n][0] - base[0]), e1 = exp2_fast(s[n][1] - base[0]);
        const float e2 = exp2_fast(s[n][2] - base[1]), e3 = exp2_fast(s[n][3] - base[1]);
        r.l[0] += e0 + e1;
        r.l[1] += e2 + e3;
        pf[n >> 1][(n & 1) * 2] = pack_bf(e0, e1);
        pf[n >> 1][(n & 1) * 2 + 1] = pack_bf(e2, e3);
    }
}

// blockIdx.x: 64 query rows.  Dynamic shared memory: flash_smem(hd, DV).
template <int DV, class Src>
__device__ __forceinline__ void flash_tile(const Src& src, const FlashShape& f, const det_seq_ref& seq) {
    extern __shared__ __align__(16) uint8_t fsm[];
    const int dqp = (f.hd + 15) & ~15, ldk = dqp + 8;
    constexpr int LDV = DV + 8;
    bf16* Q = reinterpret_cast<bf16*>(fsm);                       // [64][ldk]
    bf16* Kt = Q + FL_ROWS * ldk;                                  // [2][64][ldk]
    bf16* Vt = Kt + 2 * FL_KEYS * ldk;                             // [2][64][LDV]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    // later query rows have more keys behind them (until the window fills): start those first
    const int r0 = (gridDim.x - 1 - blockIdx.x) * FL_ROWS, nrows = min(FL_ROWS, f.M - r0);
    constexpr int NT = FL_WARPS * 32;
    pdl_trigger();
    for (int i = threadIdx.x; i < (2 * FL_KEYS * ldk + 2 * FL_KEYS * LDV) / 8; i += NT)
        reinterpret_cast<uint4*>(Kt)[i] = make_uint4(0, 0, 0, 0);
    pdl_wait();
    const int p0 = position_of(seq, r0), p_last = p0 + nrows - 1;
#pragma unroll 4
    for (int r = warp; r < FL_ROWS; r += FL_WARPS)                 // a warp per row, two neighbouring elements per lane
        for (int e = lane * 2; e < dqp; e += 64)
            *reinterpret_cast<unsigned*>(Q + r * ldk + e) = r < nrows ? src.query(r0 + r, p0 + r, e) : 0u;
    // a warp copies whole key rows; which 16-byte pieces of a row a lane takes does not depend on the row
    constexpr int PIECES = 3;
    const bf16* piece[PIECES];
    int step[PIECES];
    unsigned to[PIECES], ldt[PIECES];
#pragma unroll
    for (int j = 0; j < PIECES; j++) {
        const int v = lane + j * 32;
        piece[j] = nullptr;
        step[j] = 0;
        to[j] = ldt[j] = 0;
        if (v < src.pieces()) {
            const FlashPiece g = src.piece(v);
            piece[j] = g.p;
            step[j] = g.step;
            to[j] = smem_addr((g.value ? Vt : Kt) + g.vec * 8);
            ldt[j] = (g.value ? LDV : ldk) * 2;
        }
    }
    auto fetch = [&](int k0, int buf) {
        const int slot0 = k0 % f.cap, last = p_last - k0;         // past the last key: a copy of it, masked below
#pragma unroll
        for (int j = 0; j < PIECES; j++) {
            if (!piece[j]) continue;
            unsigned dst = to[j] + (unsigned)(buf * FL_KEYS + warp) * ldt[j];
#pragma unroll 4
            for (int k = warp; k < FL_KEYS; k += FL_WARPS, dst += FL_WARPS * ldt[j]) {
                int slot = slot0 + min(k, last);
                if (slot >= f.cap) slot = f.cap >= FL_KEYS ? slot - f.cap : slot % f.cap;
                cp_async16(dst, piece[j] + (long long)slot * step[j]);
            }
        }
        cp_async_commit();
    };
    __syncthreads();
    float o[DV / 8][4];
#pragma unroll
    for (int i = 0; i < DV / 8; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    FlashRows st{{-INFINITY, -INFINITY}, {0.0f, 0.0f}};
    const int pa = p0 + warp * 16 + (lane >> 2), pb = pa + 8;       // positions of this lane's two rows
    const int lo = first_key(p0, f.window);
    const unsigned qaddr = smem_addr(Q + (warp * 16 + (lane & 15)) * ldk + (lane >> 4) * 8);
    int buf = 0;
    fetch(lo, 0);
    for (int k0 = lo; k0 <= p_last; k0 += FL_KEYS, buf ^= 1) {
        if (k0 + FL_KEYS <= p_last) {
            fetch(k0 + FL_KEYS, buf ^ 1);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        // keys of this tile that some row of the warp sees
        const int w_first = p0 + warp * 16, w_last = w_first + 15;
        const bool seen = k0 <= w_last && (f.window <= 0 || k0 + FL_KEYS - 1 > w_first - f.window);
        if (seen) {
            float s[8][4];
#pragma unroll
            for (int i = 0; i < 8; i++) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.0f;
            const bf16* K = Kt + (size_t)buf * FL_KEYS * ldk;
            const unsigned kaddr = smem_addr(K + ((lane & 7) + ((lane >> 4) << 3)) * ldk + ((lane >> 3) & 1) * 8);
#pragma unroll 2
            for (int kk = 0; kk < dqp; kk += 16) {
                unsigned qa[4];
                ldsm4(qaddr + kk * 2, qa);
#pragma unroll
                for (int n = 0; n < 4; n++) {
                    unsigned kb[4];
                    ldsm4(kaddr + (unsigned)(n * 16 * ldk + kk) * 2, kb);
                    mma16816(s[2 * n], qa, kb[0], kb[1]);
                    mma16816(s[2 * n + 1], qa, kb[2], kb[3]);
                }
            }
            const bool edge = k0 + FL_KEYS - 1 > w_first || (f.window > 0 && k0 <= w_last - f.window);
            if (edge) {
#pragma unroll
                for (int n = 0; n < 8; n++)
#pragma unroll
                    for (int c = 0; c < 4; c++) {
                        const int j = k0 + n * 8 + (lane & 3) * 2 + (c & 1), p = c < 2 ? pa : pb;
                        if (j > p || (f.window > 0 && j <= p - f.window)) s[n][c] = -INFINITY;
                    }
            }
            unsigned pf[4][4];
            flash_softmax(st, s, o, pf);
            const bf16* V = Vt + (size_t)buf * FL_KEYS * LDV;
            const unsigned vaddr = smem_addr(V + (lane & 15) * LDV + (lane >> 4) * 8);
#pragma unroll
            for (int kk = 0; kk < 4; kk++)
#pragma unroll
                for (int n = 0; n < DV / 16; n++) {
                    unsigned vb[4];
                    ldsm4_t(vaddr + (unsigned)(kk * 16 * LDV + n * 16) * 2, vb);
                    mma16816(o[2 * n], pf[kk], vb[0], vb[1]);
                    mma16816(o[2 * n + 1], pf[kk], vb[2], vb[3]);
                }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 2; i++) {
        st.l[i] += __shfl_xor_sync(FULL, st.l[i], 1);
        st.l[i] += __shfl_xor_sync(FULL, st.l[i], 2);
        const int r = warp * 16 + (lane >> 2) + i * 8;
        if (r >= nrows) continue;
        const float inv = src.inverse(st.m[i], st.l[i]);
#pragma unroll
        for (int n = 0; n < DV / 8; n++) src.store(r0 + r, p0 + r, n * 8 + (lane & 3) * 2, o[n][i * 2] * inv, o[n][i * 2 + 1] * inv);
    }
}

}  // namespace detb
