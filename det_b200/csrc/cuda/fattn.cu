// Attention over grouped key/value heads (include/det_b200.h, det_fattn_op): rotated queries and keys, optionally rotated
// values whose sum is turned back by the query's position, one output gate per head.
//
//   k_fattn_prep    rotation; queries into a row of their own, keys and values into the sequence's cache.  One row per sequence
//                   in bfloat16 needs no such launch: k_fattn_dec rotates the row itself.
//   k_fattn_flash   a run of tokens, bfloat16: the flash loop of flash.cuh, 64 query rows of a head.
//   k_fattn_dec     few rows, bfloat16: the query heads of one key/value head are the 16 rows of an MMA tile, a CTA's four
//                   warps and further CTAs split the keys.  Bound by the bytes of the cache.
//   k_fattn_simt    fp32 activations, and heads too large for the others: a warp per query row and head, 32-bit throughout.
// CTAs that share a row leave their pieces in scratch; the one that arrives last adds them in order of the keys.
#include "flash.cuh"
#include <algorithm>

namespace detb {

struct AttnArgs {
    int heads, kv_heads, dim, vdim, rot_dims, per_kv;
    int kd, vd, ld, ldq;        // padded head sizes, elements of a cache row and of a query row
    float scale;                // times log2(e): scores in units of log 2
    int cap, M;
    const float* y;
    int ldy, q_off, k_off, v_off, gate_off;
    const float* rope_cos;
    const float* rope_sin;
    const float* vrope_cos;
    const float* vrope_sin;
    void* q;
    void* out;
    int ldo;
    float* part;                // [row][head][split][2 + vd]: maximum, sum, values
    unsigned* counters;
    int splits, per_split;
    det_seq_ref seq;
};

__device__ __forceinline__ const float* gate_of(const AttnArgs& a, int row, int h) {
    return a.gate_off < 0 ? nullptr : a.y + (size_t)row * a.ldy + a.gate_off + h;
}
// Elements v, v + 1 of a head's output: turned back by the position, gated.
template <class T>
__device__ __forceinline__ void put_out(const AttnArgs& a, int row, int pos, int h, int v, float o0, float o1) {
    if (a.vrope_cos) {
        const size_t at = (size_t)pos * (a.vdim / 2) + (v >> 1);
        const float c = a.vrope_cos[at], s = a.vrope_sin[at], u = o0;
        o0 = fmaf(u, c, o1 * s);
        o1 = fmaf(o1, c, -(u * s));
    }
    if (const float* g = gate_of(a, row, h)) {
        const float w = sigmoid_fast(*g);
        o0 *= w;
        o1 *= w;
    }
    T* out = static_cast<T*>(a.out) + (size_t)row * a.ldo + h * a.vdim + v;
    put(out, o0);
    if (v + 1 < a.vdim) put(out + 1, o1);
}

// ------------------------------------------------------------------------------------------------------ rotation
// Elements e, e + 1 of a head, zeros past its end.
__device__ __forceinline__ float2 rotated_pair(const float* x, int e, int size, int rot, const float* cs, const float* sn, int pos) {
    float u = e < size ? x[e] : 0.0f, v = e + 1 < size ? x[e + 1] : 0.0f;
    if (e < rot) {
        const size_t at = (size_t)pos * (rot / 2) + (e >> 1);
        const float c = cs[at], s = sn[at], w = u;
        u = fmaf(w, c, -(v * s));
        v = fmaf(v, c, w * s);
    }
    return make_float2(u, v);
}
__device__ __forceinline__ void put_pair(float* p, float2 v) { *reinterpret_cast<float2*>(p) = v; }
__device__ __forceinline__ void put_pair(bf16* p, float2 v) { *reinterpret_cast<unsigned*>(p) = pack_bf(v.x, v.y); }

constexpr int PREP_THREADS = 256;
template <class T>
__global__ void __launch_bounds__(PREP_THREADS) k_fattn_prep(const AttnArgs a) {
    pdl_trigger();
    pdl_wait();
    const int row = blockIdx.x, pos = position_of(a.seq, row), kp = a.kd / 2, vp = a.vd / 2;
    const int nq = a.heads * kp, nk = a.kv_heads * kp, nv = a.kv_heads * vp;
    const float* y = a.y + (size_t)row * a.ldy;
    T* q = static_cast<T*>(a.q) + (size_t)row * a.ldq;
    T* c = static_cast<T*>(slot_of(a.seq, row).cache) + (size_t)(pos % a.cap) * a.ld;
    for (int i = blockIdx.y * PREP_THREADS + threadIdx.x; i < nq + nk + nv; i += gridDim.y * PREP_THREADS) {
        if (i < nq) {
            const int h = i / kp, e = (i - h * kp) * 2;
            float2 v = rotated_pair(y + a.q_off + h * a.dim, e, a.dim, a.rot_dims, a.rope_cos, a.rope_sin, pos);
            v.x *= a.scale;
            v.y *= a.scale;
            put_pair(q + h * a.kd + e, v);
        } else if (i < nq + nk) {
            const int h = (i - nq) / kp, e = (i - nq - h * kp) * 2;
            put_pair(c + h * a.kd + e, rotated_pair(y + a.k_off + h * a.dim, e, a.dim, a.rot_dims, a.rope_cos, a.rope_sin, pos));
        } else {
            const int h = (i - nq - nk) / vp, e = (i - nq - nk - h * vp) * 2;
            put_pair(c + a.kv_heads * a.kd + h * a.vd + e,
                     rotated_pair(y + a.v_off + h * a.vdim, e, a.vdim, a.vrope_cos ? a.vdim : 0, a.vrope_cos, a.vrope_sin, pos));
        }
    }
}

// ------------------------------------------------------------------------------------------------------ a run of tokens
struct AttnFlash {
    const AttnArgs& a;
    int h, g;
    const bf16* cache;
    __device__ __forceinline__ AttnFlash(const AttnArgs& args, int head)
        : a(args), h(head), g(head / args.per_kv), cache(static_cast<const bf16*>(args.seq.one.cache)) {}
    __device__ __forceinline__ unsigned query(int row, int, int e) const {
        if (e >= a.kd) return 0;
        return *reinterpret_cast<const unsigned*>(static_cast<const bf16*>(a.q) + (size_t)row * a.ldq + h * a.kd + e);
    }
    __device__ __forceinline__ int pieces() const { return (a.kd + a.vd) / 8; }
    __device__ __forceinline__ FlashPiece piece(int v) const {
        const int kvec = a.kd / 8;
        if (v < kvec) return {cache + g * a.kd + v * 8, a.ld, v, false};
        return {cache + a.kv_heads * a.kd + g * a.vd + (v - kvec) * 8, a.ld, v - kvec, true};
    }
    __device__ __forceinline__ float inverse(float, float l) const { return 1.0f / l; }
    __device__ __forceinline__ void store(int row, int pos, int v, float o0, float o1) const {
        if (v < a.vdim) put_out<bf16>(a, row, pos, h, v, o0, o1);
    }
};
template <int DV>
__global__ void __launch_bounds__(FL_WARPS * 32, 2) k_fattn_flash(const AttnArgs a) {
    flash_tile<DV>(AttnFlash(a, blockIdx.y), FlashShape{a.kd, 0, a.cap, a.M}, a.seq);
}

// ------------------------------------------------------------------------------------------------------ pieces of a row
// True in the CTA that is the last of `splits` to arrive at a counter; its reads of the others' pieces may follow.
__device__ __forceinline__ bool last_to_arrive(unsigned* counter, int splits) {
    __shared__ unsigned last;
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) {
        last = atomicAdd(counter, 1u) == (unsigned)(splits - 1);
        if (last) *counter = 0;
    }
    __syncthreads();
    if (last) __threadfence();
    return last;
}
// A CTA adds the pieces of `nh` heads of a row from h0 on.  fac: room for nh * (splits + 1) floats.
template <class T>
__device__ __forceinline__ void merge_block(const AttnArgs& a, int row, int pos, int h0, int nh, float* fac) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5, pr = 2 + a.vd, S = a.splits;
    const float* first = a.part + ((size_t)row * a.heads + h0) * S * pr;
    for (int r = warp; r < nh; r += warps) {
        const float* p = first + (size_t)r * S * pr;
        float m = -INFINITY, l = 0.0f;
        for (int s = lane; s < S; s += 32) m = fmaxf(m, __ldcg(p + (size_t)s * pr));
        m = warp_max(m);
        for (int s = lane; s < S; s += 32) {
            const float2 ml = __ldcg(reinterpret_cast<const float2*>(p + (size_t)s * pr));
            const float f = exp2f(ml.x - m);
            fac[r * (S + 1) + s] = f;
            l = fmaf(f, ml.y, l);
        }
        l = warp_sum(l);
        if (lane == 0) fac[r * (S + 1) + S] = 1.0f / l;
    }
    __syncthreads();
    const int vp = a.vd / 2;
    for (int i = threadIdx.x; i < nh * vp; i += blockDim.x) {
        const int r = i / vp, v = (i - r * vp) * 2;
        if (v >= a.vdim) continue;
        const float* p = first + (size_t)r * S * pr + 2 + v;
        const float* f = fac + r * (S + 1);
        float o0 = 0.0f, o1 = 0.0f;
#pragma unroll 16
        for (int s = 0; s < S; s++) {
            const float2 x = __ldcg(reinterpret_cast<const float2*>(p + (size_t)s * pr));
            o0 = fmaf(f[s], x.x, o0);
            o1 = fmaf(f[s], x.y, o1);
        }
        put_out<T>(a, row, pos, h0 + r, v, o0 * f[S], o1 * f[S]);
    }
}
// A warp adds the pieces of one row and head.
template <class T>
__device__ __forceinline__ void merge_pieces(const AttnArgs& a, int row, int pos, int h) {
    const int lane = threadIdx.x & 31, pr = 2 + a.vd;
    const float* p = a.part + ((size_t)row * a.heads + h) * a.splits * pr;
    float m = -INFINITY, l = 0.0f;
    for (int s = lane; s < a.splits; s += 32) m = fmaxf(m, __ldcg(p + (size_t)s * pr));
    m = warp_max(m);
    for (int s = lane; s < a.splits; s += 32) l = fmaf(exp2f(__ldcg(p + (size_t)s * pr) - m), __ldcg(p + (size_t)s * pr + 1), l);
    const float inv = 1.0f / warp_sum(l);
    for (int v = lane * 2; v < a.vdim; v += 64) {
        float o0 = 0.0f, o1 = 0.0f;
#pragma unroll 4
        for (int s = 0; s < a.splits; s++) {
            const float f = exp2f(__ldcg(p + (size_t)s * pr) - m);
            const float2 x = __ldcg(reinterpret_cast<const float2*>(p + (size_t)s * pr + 2 + v));
            o0 = fmaf(f, x.x, o0);
            o1 = fmaf(f, x.y, o1);
        }
        put_out<T>(a, row, pos, h, v, o0 * inv, o1 * inv);
    }
}

// ------------------------------------------------------------------------------------------------------ few rows
constexpr int AD_WARPS = 4, AD_KEYS = 16, AD_STAGES = 3, AD_HEADS = 16, AT_TARGET = 2 * 148;   // AT_TARGET: CTAs of a split launch

static size_t dec_smem(int kd, int dv) {
    const int ldk = ((kd + 15) & ~15) + 8;
    const size_t ring = ((size_t)AD_HEADS * ldk + (size_t)AD_WARPS * AD_STAGES * AD_KEYS * (ldk + dv + 8)) * 2;
    return std::max({ring, (size_t)AD_WARPS * AD_HEADS * (dv + 2) * sizeof(float), (size_t)AD_HEADS * (AT_TARGET + 1) * sizeof(float)});
}

// grid (splits, kv_heads * head blocks, rows); DV = value dimensions rounded up to a multiple of 64.  `fused`: q has not been
// rotated nor k and v been cached yet (every row is its sequence's only one).
template <int DV>
__global__ void __launch_bounds__(AD_WARPS * 32) k_fattn_dec(const AttnArgs a, int fused) {
    extern __shared__ __align__(16) uint8_t asm_[];
    const int dqp = (a.kd + 15) & ~15, ldk = dqp + 8;
    constexpr int LDV = DV + 8;
    bf16* Q = reinterpret_cast<bf16*>(asm_);                                   // [16][ldk]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    bf16* Kt = Q + AD_HEADS * ldk + (size_t)warp * AD_STAGES * AD_KEYS * (ldk + LDV);   // this warp's [stage][16][ldk]
    bf16* Vt = Kt + AD_STAGES * AD_KEYS * ldk;                                  // ... and [stage][16][LDV]
    const int hblocks = (a.per_kv + AD_HEADS - 1) / AD_HEADS, g = blockIdx.y / hblocks, hb = blockIdx.y % hblocks;
    const int h0 = g * a.per_kv + hb * AD_HEADS, nh = min(AD_HEADS, a.per_kv - hb * AD_HEADS), row = blockIdx.z;
    pdl_trigger();
    // what the copies leave unwritten enters products: all of it, or the rows of queries that do not exist
    const bool pads = dqp != a.kd || DV != a.vd;
    const int words = (AD_HEADS * ldk + (pads ? AD_WARPS * AD_STAGES * AD_KEYS * (ldk + LDV) : 0)) / 8;
    for (int i = threadIdx.x; i < words; i += AD_WARPS * 32) reinterpret_cast<uint4*>(asm_)[i] = make_uint4(0, 0, 0, 0);
    __syncthreads();
    pdl_wait();
    const int pos = position_of(a.seq, row);
    const int lo = blockIdx.x * a.per_split, hi = min(pos + 1, lo + a.per_split);
    bf16* cache = static_cast<bf16*>(slot_of(a.seq, row).cache);
    if (fused) {
        const float* y = a.y + (size_t)row * a.ldy;
        const int kp = a.kd / 2, vp = a.vd / 2;
        bf16* c = cache + (size_t)pos * a.ld;
        const int own = hi == pos + 1 && lo < hi ? kp + vp : 0;               // the CTAs that read the new key also cache it
        for (int i = threadIdx.x; i < nh * kp + own; i += AD_WARPS * 32) {
            if (i < nh * kp) {
                const int h = i / kp, e = (i - h * kp) * 2;
                float2 v = rotated_pair(y + a.q_off + (h0 + h) * a.dim, e, a.dim, a.rot_dims, a.rope_cos, a.rope_sin, pos);
                put_pair(Q + h * ldk + e, make_float2(v.x * a.scale, v.y * a.scale));
            } else if (i < nh * kp + kp) {
                const int e = (i - nh * kp) * 2;
                put_pair(c + g * a.kd + e, rotated_pair(y + a.k_off + g * a.dim, e, a.dim, a.rot_dims, a.rope_cos, a.rope_sin, pos));
            } else {
                const int e = (i - nh * kp - kp) * 2;
                put_pair(c + a.kv_heads * a.kd + g * a.vd + e,
                         rotated_pair(y + a.v_off + g * a.vdim, e, a.vdim, a.vrope_cos ? a.vdim : 0, a.vrope_cos, a.vrope_sin, pos));
            }
        }
    } else {
        const bf16* q = static_cast<const bf16*>(a.q) + (size_t)row * a.ldq + (size_t)h0 * a.kd;
        for (int i = threadIdx.x; i < nh * (a.kd / 8); i += AD_WARPS * 32) {
            const int h = i / (a.kd / 8), v = i % (a.kd / 8);
            *reinterpret_cast<uint4*>(Q + h * ldk + v * 8) = *reinterpret_cast<const uint4*>(q + h * a.kd + v * 8);
        }
    }
    __syncthreads();
    const int kvec = a.kd / 8, tvec = kvec + a.vd / 8;
    auto fetch = [&](int k0, int stage) {
        if (k0 < hi)
            for (int v = lane; v < tvec; v += 32) {
                const bool val = v >= kvec;
                const bf16* src = cache + (val ? a.kv_heads * a.kd + g * a.vd + (v - kvec) * 8 : g * a.kd + v * 8);
                unsigned dst = smem_addr(val ? Vt + stage * AD_KEYS * LDV + (v - kvec) * 8 : Kt + stage * AD_KEYS * ldk + v * 8);
                const unsigned step = (val ? LDV : ldk) * 2;
#pragma unroll
                for (int k = 0; k < AD_KEYS; k++, dst += step) cp_async16(dst, src + (size_t)min(k0 + k, hi - 1) * a.ld);
            }
        cp_async_commit();
    };
    float o[DV / 8][4];
#pragma unroll
    for (int i = 0; i < DV / 8; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    FlashRows st{{-INFINITY, -INFINITY}, {0.0f, 0.0f}};
    const unsigned qaddr = smem_addr(Q + (lane & 15) * ldk + (lane >> 4) * 8);
    constexpr int STEP = AD_WARPS * AD_KEYS;
    int k0 = lo + warp * AD_KEYS;
#pragma unroll
    for (int s = 0; s < AD_STAGES - 1; s++) fetch(k0 + s * STEP, s);
    for (int stage = 0; k0 < hi; k0 += STEP, stage = stage + 1 == AD_STAGES ? 0 : stage + 1) {
        fetch(k0 + (AD_STAGES - 1) * STEP, stage == 0 ? AD_STAGES - 1 : stage - 1);
        cp_async_wait<AD_STAGES - 1>();
        __syncwarp();
        float s[2][4];
#pragma unroll
        for (int i = 0; i < 2; i++) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.0f;
        const unsigned kaddr = smem_addr(Kt + stage * AD_KEYS * ldk + ((lane & 7) + ((lane >> 4) << 3)) * ldk + ((lane >> 3) & 1) * 8);
#pragma unroll 4
        for (int kk = 0; kk < dqp; kk += 16) {
            unsigned qa[4], kb[4];
            ldsm4(qaddr + kk * 2, qa);
            ldsm4(kaddr + kk * 2, kb);
            mma16816(s[0], qa, kb[0], kb[1]);
            mma16816(s[1], qa, kb[2], kb[3]);
        }
        if (k0 + AD_KEYS > hi) {
#pragma unroll
            for (int n = 0; n < 2; n++)
#pragma unroll
                for (int c = 0; c < 4; c++)
                    if (k0 + n * 8 + (lane & 3) * 2 + (c & 1) >= hi) s[n][c] = -INFINITY;
        }
        unsigned pf[1][4];
        flash_softmax(st, s, o, pf);
        const unsigned vaddr = smem_addr(Vt + stage * AD_KEYS * LDV + (lane & 15) * LDV + (lane >> 4) * 8);
#pragma unroll
        for (int n = 0; n < DV / 16; n++) {
            unsigned vb[4];
            ldsm4_t(vaddr + n * 32, vb);
            mma16816(o[2 * n], pf[0], vb[0], vb[1]);
            mma16816(o[2 * n + 1], pf[0], vb[2], vb[3]);
        }
        __syncwarp();
    }
    cp_async_wait<0>();
    __syncthreads();
    // the warps' pieces: [warp][head][DV] values, then [warp][head] maximum and sum
    float* po = reinterpret_cast<float*>(asm_);
    float* ml = po + AD_WARPS * AD_HEADS * DV;
#pragma unroll
    for (int i = 0; i < 2; i++) {
        st.l[i] += __shfl_xor_sync(FULL, st.l[i], 1);
        st.l[i] += __shfl_xor_sync(FULL, st.l[i], 2);
        const int r = (lane >> 2) + i * 8, at = warp * AD_HEADS + r;
        if ((lane & 3) == 0) {
            ml[at * 2] = st.m[i];
            ml[at * 2 + 1] = st.l[i];
        }
#pragma unroll
        for (int n = 0; n < DV / 8; n++)
            *reinterpret_cast<float2*>(po + (size_t)at * DV + n * 8 + (lane & 3) * 2) = make_float2(o[n][i * 2], o[n][i * 2 + 1]);
    }
    __syncthreads();
    const int vp = a.vd / 2;
    for (int i = threadIdx.x; i < nh * vp; i += AD_WARPS * 32) {
        const int r = i / vp, v = (i - r * vp) * 2;
        float m = -INFINITY, l = 0.0f, o0 = 0.0f, o1 = 0.0f;
#pragma unroll
        for (int w = 0; w < AD_WARPS; w++) m = fmaxf(m, ml[(w * AD_HEADS + r) * 2]);
        const float base = m == -INFINITY ? 0.0f : m;              // a piece without keys
#pragma unroll
        for (int w = 0; w < AD_WARPS; w++) {
            const int at = w * AD_HEADS + r;
            const float f = exp2f(ml[at * 2] - base);
            const float2 x = *reinterpret_cast<const float2*>(po + (size_t)at * DV + v);
            l = fmaf(f, ml[at * 2 + 1], l);
            o0 = fmaf(f, x.x, o0);
            o1 = fmaf(f, x.y, o1);
        }
        if (a.splits == 1) {
            if (v < a.vdim) put_out<bf16>(a, row, pos, h0 + r, v, o0 / l, o1 / l);
        } else {
            float* p = a.part + (((size_t)row * a.heads + h0 + r) * a.splits + blockIdx.x) * (2 + a.vd);
            if (v == 0) *reinterpret_cast<float2*>(p) = make_float2(m, l);
            *reinterpret_cast<float2*>(p + 2 + v) = make_float2(o0, o1);
        }
    }
    if (a.splits == 1 || !last_to_arrive(a.counters + (size_t)row * gridDim.y + blockIdx.y, a.splits)) return;
    merge_block<bf16>(a, row, pos, h0, nh, reinterpret_cast<float*>(asm_));
}

// ------------------------------------------------------------------------------------------------------ 32-bit, any size
constexpr int AS_WARPS = 8;

__device__ __forceinline__ float2 load_pair(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 load_pair(const bf16* p) {
    const unsigned v = *reinterpret_cast<const unsigned*>(p);
    return make_float2(bf_lo(v), bf_hi(v));
}

// grid (splits, heads / 8, rows); NP: pairs of a head's elements per lane (64 * NP >= kd, vd)
template <class T, int NP>
__global__ void __launch_bounds__(AS_WARPS * 32) k_fattn_simt(const AttnArgs a) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, row = blockIdx.z, h = blockIdx.y * AS_WARPS + warp;
    pdl_trigger();
    pdl_wait();
    const int pos = position_of(a.seq, row);
    const int lo = blockIdx.x * a.per_split, hi = min(pos + 1, lo + a.per_split);
    if (h < a.heads) {
        const int g = h / a.per_kv;
        const T* keys = static_cast<const T*>(slot_of(a.seq, row).cache) + (size_t)g * a.kd;
        const T* values = static_cast<const T*>(slot_of(a.seq, row).cache) + (size_t)a.kv_heads * a.kd + (size_t)g * a.vd;
        const T* qr = static_cast<const T*>(a.q) + (size_t)row * a.ldq + (size_t)h * a.kd;
        float2 q[NP], acc[NP];
#pragma unroll
        for (int i = 0; i < NP; i++) {
            const int e = (i * 32 + lane) * 2;
            q[i] = e < a.kd ? load_pair(qr + e) : make_float2(0.0f, 0.0f);
            acc[i] = make_float2(0.0f, 0.0f);
        }
        float m = -INFINITY, l = 0.0f;
        for (int k = lo; k < hi; k += 4) {
            float s[4];
#pragma unroll
            for (int j = 0; j < 4; j++) {
                const T* key = keys + (size_t)min(k + j, hi - 1) * a.ld;
                s[j] = 0.0f;
#pragma unroll
                for (int i = 0; i < NP; i++) {
                    const int e = (i * 32 + lane) * 2;
                    if (e >= a.kd) continue;
                    const float2 c = load_pair(key + e);
                    s[j] = fmaf(q[i].x, c.x, s[j]);
                    s[j] = fmaf(q[i].y, c.y, s[j]);
                }
            }
#pragma unroll
            for (int j = 0; j < 4; j++) {
                s[j] = warp_sum(s[j]);
                if (k + j >= hi) s[j] = -INFINITY;
            }
            const float mn = fmaxf(fmaxf(m, fmaxf(s[0], s[1])), fmaxf(s[2], s[3]));
            const float f = exp2f(m - mn);
            m = mn;
            l *= f;
#pragma unroll
            for (int i = 0; i < NP; i++) {
                acc[i].x *= f;
                acc[i].y *= f;
            }
#pragma unroll
            for (int j = 0; j < 4; j++) {
                const T* val = values + (size_t)min(k + j, hi - 1) * a.ld;
                const float p = exp2f(s[j] - m);
                l += p;
#pragma unroll
                for (int i = 0; i < NP; i++) {
                    const int e = (i * 32 + lane) * 2;
                    if (e >= a.vd) continue;
                    const float2 c = load_pair(val + e);
                    acc[i].x = fmaf(p, c.x, acc[i].x);
                    acc[i].y = fmaf(p, c.y, acc[i].y);
                }
            }
        }
        float* p = a.part + (((size_t)row * a.heads + h) * a.splits + blockIdx.x) * (2 + a.vd);
        if (a.splits > 1 && lane == 0) *reinterpret_cast<float2*>(p) = make_float2(m, l);
#pragma unroll
        for (int i = 0; i < NP; i++) {
            const int e = (i * 32 + lane) * 2;
            if (a.splits > 1) {
                if (e < a.vd) *reinterpret_cast<float2*>(p + 2 + e) = acc[i];
            } else if (e < a.vdim) {
                put_out<T>(a, row, pos, h, e, acc[i].x / l, acc[i].y / l);
            }
        }
    }
    if (a.splits == 1 || !last_to_arrive(a.counters + (size_t)row * gridDim.y + blockIdx.y, a.splits)) return;
    if (h < a.heads) merge_pieces<T>(a, row, pos, h);
}

// ------------------------------------------------------------------------------------------------------ host side
static bool takes_flash(const det_fattn_op& op, const AttnArgs& a) {
    const int dv = (a.vd + 63) / 64 * 64;
    return op.dtype == DET_BF16 && !op.seq.table && !op.seq.pos && op.M >= 32 && !(float_flags() & 8) && a.vd <= 256 &&
           a.kd + a.vd <= 768 && flash_smem(a.kd, dv) <= 220 * 1024;
}
static bool takes_dec(const det_fattn_op& op, const AttnArgs& a) {
    return op.dtype == DET_BF16 && !(float_flags() & 8) && a.vd <= 256 && dec_smem(a.kd, (a.vd + 63) / 64 * 64) <= 220 * 1024;
}
// Calls whose rows k_fattn_dec rotates and caches itself: one row per sequence.
static bool rotates_itself(const det_fattn_op& op, const AttnArgs& a) {
    return (op.seq.table || op.M == 1) && takes_dec(op, a) && !takes_flash(op, a);
}
// Key ranges per row: enough CTAs to fill the device, at least 64 keys each.
static void plan(AttnArgs& a, int blocks, int max_pos, int target) {
    const long long ctas = (long long)a.M * blocks;
    const int keys = max_pos + 1;
    int s = (int)std::min<long long>((keys + 63) / 64, target / ctas);
    int n = 0;
    unsigned* counters = fsplit_counters(&n);
    if (ctas > n) s = 1;
    s = std::max(1, s);
    a.per_split = ((keys + s - 1) / s + 63) / 64 * 64;
    a.splits = (keys + a.per_split - 1) / a.per_split;
    a.counters = counters;
}
template <int DV>
static void launch_flash(const AttnArgs& a, cudaStream_t q) {
    const size_t smem = flash_smem(a.kd, DV);
    static size_t configured = 0;
    if (smem > configured) {
        DETB_CUDA_OK(cudaFuncSetAttribute(k_fattn_flash<DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        configured = smem;
    }
    launch_plain(k_fattn_flash<DV>, dim3((a.M + FL_ROWS - 1) / FL_ROWS, a.heads), dim3(FL_WARPS * 32), smem, q, a);
}
template <int DV>
static void launch_dec(AttnArgs a, int max_pos, bool fused, cudaStream_t q) {
    const size_t smem = dec_smem(a.kd, DV);
    static size_t configured = 0;
    if (smem > configured) {
        DETB_CUDA_OK(cudaFuncSetAttribute(k_fattn_dec<DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        configured = smem;
    }
    const int blocks = a.kv_heads * ((a.per_kv + AD_HEADS - 1) / AD_HEADS);
    plan(a, blocks, max_pos, AT_TARGET / 2);
    launch_pdl(k_fattn_dec<DV>, dim3(a.splits, blocks, a.M), dim3(AD_WARPS * 32), smem, q, 1, a, fused ? 1 : 0);
}
template <class T>
static void launch_simt(AttnArgs a, int max_pos, cudaStream_t q) {
    const int blocks = (a.heads + AS_WARPS - 1) / AS_WARPS, np = (std::max(a.kd, a.vd) + 63) / 64;
    plan(a, blocks, max_pos, AT_TARGET);
    const dim3 grid(a.splits, blocks, a.M), block(AS_WARPS * 32);
    if (np <= 2) launch_pdl(k_fattn_simt<T, 2>, grid, block, 0, q, 1, a);
    else if (np <= 4) launch_pdl(k_fattn_simt<T, 4>, grid, block, 0, q, 1, a);
    else if (np <= 8) launch_pdl(k_fattn_simt<T, 8>, grid, block, 0, q, 1, a);
    else launch_pdl(k_fattn_simt<T, 16>, grid, block, 0, q, 1, a);
}

static AttnArgs attn_args(const det_fattn_op* op) {
    DETB_REQUIRE(op->heads > 0 && op->kv_heads > 0 && op->heads % op->kv_heads == 0 && op->dim > 0 && op->vdim > 0 && op->cap > 0,
                 "attention: bad sizes");
    DETB_REQUIRE(op->dim <= 1024 && op->vdim <= 1024, "attention: the head is too large");
    DETB_REQUIRE(op->rot_dims % 2 == 0 && op->rot_dims <= op->dim && (!op->vrope_cos || op->vdim % 2 == 0), "attention: bad rotation");
    DETB_REQUIRE(op->M <= 65535 && op->kv_heads <= 4096, "attention: too many rows");
    AttnArgs a{};
    a.heads = op->heads; a.kv_heads = op->kv_heads; a.dim = op->dim; a.vdim = op->vdim; a.rot_dims = op->rot_dims;
    a.per_kv = op->heads / op->kv_heads;
    a.kd = round8(op->dim); a.vd = round8(op->vdim);
    a.ld = det_f_attn_ld(op->kv_heads, op->dim, op->vdim);
    a.ldq = det_f_attn_q_ld(op->heads, op->dim);
    a.scale = op->scale * 1.4426950408889634f;
    a.cap = op->cap; a.M = op->M;
    a.y = op->y; a.ldy = op->ldy; a.q_off = op->q_off; a.k_off = op->k_off; a.v_off = op->v_off; a.gate_off = op->gate_off;
    a.rope_cos = op->rope_cos; a.rope_sin = op->rope_sin; a.vrope_cos = op->vrope_cos; a.vrope_sin = op->vrope_sin;
    a.q = op->q; a.out = op->out; a.ldo = op->ldo;
    a.part = static_cast<float*>(op->scratch);
    a.seq = op->seq;
    return a;
}

}  // namespace detb

using namespace detb;

extern "C" {

int det_f_attn_ld(int kv_heads, int dim, int vdim) { return kv_heads * (round8(dim) + round8(vdim)); }
int det_f_attn_q_ld(int heads, int dim) { return heads * round8(dim); }
// A launch with pieces has at most AT_TARGET CTAs, each with up to 16 heads.
size_t det_f_attn_scratch_bytes(int vdim) { return (size_t)AT_TARGET * AD_HEADS * (2 + round8(vdim)) * sizeof(float); }

void det_f_attn_prep(const det_fattn_op* op, cudaStream_t st) {
    const AttnArgs a = attn_args(op);
    if (op->M <= 0 || rotates_itself(*op, a)) return;
    const int pairs = (a.heads + a.kv_heads) * a.kd / 2 + a.kv_heads * a.vd / 2;
    const int pieces = std::max(1, std::min((pairs + PREP_THREADS - 1) / PREP_THREADS, 4 * sm_count() / op->M));
    if (op->dtype == DET_BF16) launch_pdl(k_fattn_prep<bf16>, dim3(op->M, pieces), dim3(PREP_THREADS), 0, queue_of(st), 1, a);
    else launch_pdl(k_fattn_prep<float>, dim3(op->M, pieces), dim3(PREP_THREADS), 0, queue_of(st), 1, a);
}

void det_f_attn(const det_fattn_op* op, cudaStream_t st) {
    const AttnArgs a = attn_args(op);
    if (op->M <= 0) return;
    DETB_REQUIRE(op->max_pos < op->cap, "attention: positions beyond the cache");
    cudaStream_t q = queue_of(st);
    const int dv = (a.vd + 63) / 64;
    if (takes_flash(*op, a)) {
        if (dv == 1) launch_flash<64>(a, q);
        else if (dv == 2) launch_flash<128>(a, q);
        else if (dv == 3) launch_flash<192>(a, q);
        else launch_flash<256>(a, q);
    } else if (takes_dec(*op, a)) {
        const bool fused = rotates_itself(*op, a);
        if (dv == 1) launch_dec<64>(a, op->max_pos, fused, q);
        else if (dv == 2) launch_dec<128>(a, op->max_pos, fused, q);
        else if (dv == 3) launch_dec<192>(a, op->max_pos, fused, q);
        else launch_dec<256>(a, op->max_pos, fused, q);
    } else if (op->dtype == DET_BF16) {
        launch_simt<bf16>(a, op->max_pos, q);
    } else {
        launch_simt<float>(a, op->max_pos, q);
    }
}

}  // extern "C"
