// Latent attention (include/det_b200.h, det_flatent_op): one cached latent row per position for all heads, sliding window,
// softmax with a sink, output gate.
//
// Two forms of the same sums:
//   absorbed (decode, and everything with fp32 activations): scores and values are taken in the latent space, so the cache
//     row is key and value at once.  k_latent_absorb: q W_uk per head; k_latent_scores: a warp per head walks a range of
//     keys staged in shared memory, online softmax; k_latent_out merges the ranges, adds the sink, applies W_uv and the gate.
//   expanded (a run of tokens with bfloat16 activations): keys and values of the cached rows are multiplied out by the
//     tensor-core GEMM, then k_latent_flash computes 64 query rows of a head against 64-key tiles with bfloat16 MMAs.
#include "flash.cuh"
#include <algorithm>
#include <cmath>
#include <type_traits>

namespace detb {

struct LatentArgs {
    int heads, dim, rot_dim, rot_dims, vdim, q_rank, kv_rank;
    int rp, ld;                 // offset of the rotated part in a cache row, elements of a cache row
    int window;
    float scale;
    int cap, M;
    const float* y;
    int ldy, dq_off, dkv_off, gate_off;
    const float* dq_norm;
    const float* dkv_norm;
    float eps;
    const float* rope_cos;
    const float* rope_sin;
    void* cq;
    int ldcq;
    const float* q;
    int ldq;
    const bf16* wkv;
    int ldw;
    const float* sink;
    void* out;
    int ldo;
    float* qa;                  // [M][heads][ld] absorbed queries, times scale
    float* part;                // [M][heads][splits][kv_rank + 2]: m, l, then the weighted latent sum
    int splits, per_split;
    const bf16* kv;             // expanded [slot][heads * dim | heads * vdim]
    int ldkv;
    det_seq_ref seq;
};

// element e of the rotated part of a head at `pos` (pairs (2i, 2i + 1) of the first rot_dims elements)
__device__ __forceinline__ float rotated(const float* x, int e, int pos, const LatentArgs& a) {
    if (e >= a.rot_dims) return x[e];
    const size_t at = (size_t)pos * (a.rot_dims / 2) + (e >> 1);
    const float c = a.rope_cos[at], s = a.rope_sin[at];
    return (e & 1) ? fmaf(x[e], c, x[e - 1] * s) : fmaf(x[e], c, -(x[e + 1] * s));
}

// ------------------------------------------------------------------------------------------------------ rows into cq and cache
template <class T>
__global__ void __launch_bounds__(256) k_latent_prep(const LatentArgs a) {
    __shared__ float sh[32];
    pdl_trigger();
    pdl_wait();
    const int row = blockIdx.x, pos = position_of(a.seq, row);
    const float* dq = a.y + (size_t)row * a.ldy + a.dq_off;
    const float* dkv = a.y + (size_t)row * a.ldy + a.dkv_off;
    float s = 0.0f, s2 = 0.0f;
    for (int i = threadIdx.x; i < a.q_rank; i += 256) s = fmaf(dq[i], dq[i], s);
    for (int i = threadIdx.x; i < a.kv_rank; i += 256) s2 = fmaf(dkv[i], dkv[i], s2);
    const float rq = 1.0f / sqrtf(block_sum(s, sh) / (float)a.q_rank + a.eps);
    const float rk = 1.0f / sqrtf(block_sum(s2, sh) / (float)a.kv_rank + a.eps);
    T* cq = static_cast<T*>(a.cq) + (size_t)row * a.ldcq;
    for (int i = threadIdx.x; i < a.q_rank; i += 256) put(cq + i, dq[i] * rq * a.dq_norm[i]);
    T* c = static_cast<T*>(slot_of(a.seq, row).cache) + (size_t)(pos % a.cap) * a.ld;
    for (int i = threadIdx.x; i < a.kv_rank; i += 256) put(c + i, dkv[i] * rk * a.dkv_norm[i]);
    for (int i = threadIdx.x; i < a.rot_dim; i += 256) put(c + a.rp + i, rotated(dkv + a.kv_rank, i, pos, a));
}

// ------------------------------------------------------------------------------------------------------ absorbed form
constexpr int AB_ROWS = 8;       // query rows per CTA
constexpr int AB_COLS = 64;      // latent columns per CTA: two per lane; four warps share the head's dimensions
__global__ void __launch_bounds__(128) k_latent_absorb(const LatentArgs a) {
    extern __shared__ __align__(16) float qs[];      // [AB_ROWS][dim], then the warps' partial sums [4][AB_ROWS][AB_COLS]
    const int h = blockIdx.x, r0 = blockIdx.z * AB_ROWS, nr = min(AB_ROWS, a.M - r0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* sums = qs + AB_ROWS * a.dim;
    pdl_trigger();
    pdl_wait();
    const int hd = a.dim + a.rot_dim;
    for (int i = threadIdx.x; i < nr * a.dim; i += 128) {
        const int r = i / a.dim, d = i % a.dim;
        qs[i] = a.q[(size_t)(r0 + r) * a.ldq + h * hd + d] * a.scale;
    }
    __syncthreads();
    const int c = blockIdx.y * AB_COLS + lane * 2;
    const bf16* w = a.wkv + (size_t)h * a.dim * a.ldw + min(c, a.rp - 2);      // rows padded with zeros to a multiple of 8
    auto run = [&](auto rows) {
        constexpr int R = decltype(rows)::value;
        float acc[R][2];
#pragma unroll
        for (int r = 0; r < R; r++) acc[r][0] = acc[r][1] = 0.0f;
#pragma unroll 16
        for (int d = warp; d < a.dim; d += 4) {
            const unsigned b = __ldg(reinterpret_cast<const unsigned*>(w + (size_t)d * a.ldw));
            const float w0 = bf_lo(b), w1 = bf_hi(b);
#pragma unroll
            for (int r = 0; r < R; r++) {
                const float q = qs[r * a.dim + d];
                acc[r][0] = fmaf(q, w0, acc[r][0]);
                acc[r][1] = fmaf(q, w1, acc[r][1]);
            }
        }
#pragma unroll
        for (int r = 0; r < R; r++) *reinterpret_cast<float2*>(sums + (warp * AB_ROWS + r) * AB_COLS + lane * 2) = make_float2(acc[r][0], acc[r][1]);
    };
    if (nr == 1) run(std::integral_constant<int, 1>{});
    else run(std::integral_constant<int, AB_ROWS>{});
    __syncthreads();
    for (int i = threadIdx.x; i < nr * AB_COLS; i += 128) {
        const int r = i / AB_COLS, cc = i % AB_COLS, col = blockIdx.y * AB_COLS + cc;
        if (col < a.rp) {
            float v = 0.0f;
#pragma unroll
            for (int k = 0; k < 4; k++) v += sums[(k * AB_ROWS + r) * AB_COLS + cc];
            a.qa[((size_t)(r0 + r) * a.heads + h) * a.ld + col] = v;
        }
    }
    if (blockIdx.y == 0)
        for (int i = threadIdx.x; i < nr * (a.ld - a.rp); i += 128) {
            const int r = i / (a.ld - a.rp), e = i % (a.ld - a.rp);
            const float* q = a.q + (size_t)(r0 + r) * a.ldq + h * hd + a.dim;
            a.qa[((size_t)(r0 + r) * a.heads + h) * a.ld + a.rp + e] =
                e < a.rot_dim ? rotated(q, e, position_of(a.seq, r0 + r), a) * a.scale : 0.0f;
        }
}

constexpr int LS_WARPS = 8, LS_KEYS = 16;     // heads per CTA, keys per staged tile

__device__ __forceinline__ void pair_of(const float* p, float& x, float& y) {
    const float2 v = *reinterpret_cast<const float2*>(p);
    x = v.x;
    y = v.y;
}
__device__ __forceinline__ void pair_of(const bf16* p, float& x, float& y) {
    const unsigned v = *reinterpret_cast<const unsigned*>(p);
    x = bf_lo(v);
    y = bf_hi(v);
}

// NP: pairs of elements per lane (64 * NP >= ld)
template <class T, int NP>
__global__ void __launch_bounds__(LS_WARPS * 32) k_latent_scores(const LatentArgs a) {
    extern __shared__ __align__(16) uint8_t lsm[];
    T* tile = reinterpret_cast<T*>(lsm);              // [2][LS_KEYS][64 * NP]
    constexpr int LDT = 64 * NP, VEC = 16 / sizeof(T);
    const int row = blockIdx.z, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int h = blockIdx.y * LS_WARPS + warp;
    pdl_trigger();
    // columns past a row's end stay zero; so do rows before their first use
    for (int i = threadIdx.x; i < 2 * LS_KEYS * LDT / VEC; i += LS_WARPS * 32) reinterpret_cast<uint4*>(tile)[i] = make_uint4(0, 0, 0, 0);
    pdl_wait();
    const int pos = position_of(a.seq, row);
    const int lo = first_key(pos, a.window) + blockIdx.x * a.per_split, hi = min(pos + 1, lo + a.per_split);
    const T* cache = static_cast<const T*>(slot_of(a.seq, row).cache);
    float q[NP][2], acc[NP][2];
#pragma unroll
    for (int i = 0; i < NP; i++) {
        const int e = (i * 32 + lane) * 2;
        q[i][0] = q[i][1] = acc[i][0] = acc[i][1] = 0.0f;
        if (h < a.heads && e < a.ld) pair_of(a.qa + ((size_t)row * a.heads + h) * a.ld + e, q[i][0], q[i][1]);
    }
    float m = -INFINITY, l = 0.0f;
    const int vecs = a.ld / VEC;
    auto fetch = [&](int k0, int buf) {
        const int slot0 = k0 % a.cap;
        for (int k = warp; k < LS_KEYS && k0 + k < hi; k += LS_WARPS) {      // a warp copies a row
            int slot = slot0 + k;
            while (slot >= a.cap) slot -= a.cap;
            const T* src = cache + (size_t)slot * a.ld;
            const T* dst = tile + ((size_t)buf * LS_KEYS + k) * LDT;
            for (int v = lane; v < vecs; v += 32)
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_addr(dst + v * VEC)), "l"(src + v * VEC) : "memory");
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    __syncthreads();
    int buf = 0;
    if (lo < hi) fetch(lo, 0);
    for (int k0 = lo; k0 < hi; k0 += LS_KEYS, buf ^= 1) {
        if (k0 + LS_KEYS < hi) {
            fetch(k0 + LS_KEYS, buf ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        if (h < a.heads) {
            const T* t = tile + (size_t)buf * LS_KEYS * LDT;
            for (int k = 0; k < LS_KEYS && k0 + k < hi; k += 4) {
                float c[4][NP][2], s[4];
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    s[j] = 0.0f;
#pragma unroll
                    for (int i = 0; i < NP; i++) {
                        pair_of(t + (size_t)(k + j) * LDT + (i * 32 + lane) * 2, c[j][i][0], c[j][i][1]);
                        s[j] = fmaf(q[i][0], c[j][i][0], s[j]);
                        s[j] = fmaf(q[i][1], c[j][i][1], s[j]);
                    }
                }
                // four sums over the warp: fold two keys per half-warp, then one per quarter
                const bool up = lane & 16;
                float x = (up ? s[1] : s[0]) + __shfl_xor_sync(FULL, up ? s[0] : s[1], 16);
                float z = (up ? s[3] : s[2]) + __shfl_xor_sync(FULL, up ? s[2] : s[3], 16);
                const bool up2 = lane & 8;
                x = (up2 ? z : x) + __shfl_xor_sync(FULL, up2 ? x : z, 8);
                x += __shfl_xor_sync(FULL, x, 4);
                x += __shfl_xor_sync(FULL, x, 2);
                x += __shfl_xor_sync(FULL, x, 1);
                s[0] = __shfl_sync(FULL, x, 0);
                s[1] = __shfl_sync(FULL, x, 16);
                s[2] = __shfl_sync(FULL, x, 8);
                s[3] = __shfl_sync(FULL, x, 24);
#pragma unroll
                for (int j = 1; j < 4; j++)
                    if (k0 + k + j >= hi) s[j] = -INFINITY;
                const float mn = fmaxf(fmaxf(m, fmaxf(s[0], s[1])), fmaxf(s[2], s[3]));
                if (mn > m) {                     // the same in every lane
                    const float f = expf(m - mn);
                    l *= f;
#pragma unroll
                    for (int i = 0; i < NP; i++) {
                        acc[i][0] *= f;
                        acc[i][1] *= f;
                    }
                    m = mn;
                }
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    const float p = expf(s[j] - m);
                    l += p;
#pragma unroll
                    for (int i = 0; i < NP; i++) {
                        acc[i][0] = fmaf(p, c[j][i][0], acc[i][0]);
                        acc[i][1] = fmaf(p, c[j][i][1], acc[i][1]);
                    }
                }
            }
        }
        __syncthreads();
    }
    if (h >= a.heads) return;
    float* out = a.part + (((size_t)row * a.heads + h) * a.splits + blockIdx.x) * (a.kv_rank + 2);
    if (lane == 0) {
        out[0] = m;
        out[1] = l;
    }
#pragma unroll
    for (int i = 0; i < NP; i++) {
        const int e = (i * 32 + lane) * 2;
        if (e < a.kv_rank) out[2 + e] = acc[i][0];
        if (e + 1 < a.kv_rank) out[3 + e] = acc[i][1];
    }
}

constexpr int LO_V = 32;      // value dimensions per CTA
template <class T>
__global__ void __launch_bounds__(256) k_latent_out(const LatentArgs a) {
    extern __shared__ __align__(16) float osm[];
    float* ol = osm;                               // [kv_rank rounded up to 8]
    float* fac = osm + ((a.kv_rank + 7) & ~7);     // [splits]
    __shared__ float total;
    const int h = blockIdx.x, row = blockIdx.z, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    pdl_trigger();
    pdl_wait();
    const int pr = a.kv_rank + 2;
    const float* part = a.part + ((size_t)row * a.heads + h) * a.splits * pr;
    if (warp == 0) {
        float m = a.sink ? a.sink[h] : -INFINITY;
        for (int s = lane; s < a.splits; s += 32) m = fmaxf(m, part[(size_t)s * pr]);
        m = warp_max(m);
        float l = 0.0f;
        for (int s = lane; s < a.splits; s += 32) {
            const float f = expf(part[(size_t)s * pr] - m);
            fac[s] = f;
            l = fmaf(f, part[(size_t)s * pr + 1], l);
        }
        l = warp_sum(l);
        if (a.sink) l += expf(a.sink[h] - m);
        if (lane == 0) total = 1.0f / l;
    }
    __syncthreads();
    const float inv = total;
    for (int r = threadIdx.x; r < ((a.kv_rank + 7) & ~7); r += 256) {
        float o = 0.0f;
        if (r < a.kv_rank) {
#pragma unroll 8
            for (int s = 0; s < a.splits; s++) o = fmaf(fac[s], part[(size_t)s * pr + 2 + r], o);
        }
        ol[r] = o * inv;
    }
    __syncthreads();
    const float* gate = a.y + (size_t)row * a.ldy + a.gate_off + h * a.vdim;
    T* out = static_cast<T*>(a.out) + (size_t)row * a.ldo + h * a.vdim;
    const bf16* wv = a.wkv + (size_t)(a.heads * a.dim + h * a.vdim) * a.ldw;
    const int v1 = min(a.vdim, (int)(blockIdx.y + 1) * LO_V);
    for (int v = blockIdx.y * LO_V + warp; v < v1; v += 8) {
        float s = 0.0f;
        for (int c = lane * 8; c < a.kv_rank; c += 256) {
            const uint4 b = *reinterpret_cast<const uint4*>(wv + (size_t)v * a.ldw + c);
            const float4 x = *reinterpret_cast<const float4*>(ol + c), y = *reinterpret_cast<const float4*>(ol + c + 4);
            s = fmaf(bf_lo(b.x), x.x, s);
            s = fmaf(bf_hi(b.x), x.y, s);
            s = fmaf(bf_lo(b.y), x.z, s);
            s = fmaf(bf_hi(b.y), x.w, s);
            s = fmaf(bf_lo(b.z), y.x, s);
            s = fmaf(bf_hi(b.z), y.y, s);
            s = fmaf(bf_lo(b.w), y.z, s);
            s = fmaf(bf_hi(b.w), y.w, s);
        }
        s = warp_sum(s);
        if (lane == 0) put(out + v, s * sigmoid_fast(gate[v]));
    }
}

// ------------------------------------------------------------------------------------------------------ expanded form
// One head of the expanded form for the flash loop: keys are [expanded part | rotated part of the cache row].
struct LatentFlash {
    const LatentArgs& a;
    int h;
    const bf16* cache;
    __device__ __forceinline__ LatentFlash(const LatentArgs& args, int head)
        : a(args), h(head), cache(static_cast<const bf16*>(args.seq.one.cache)) {}
    __device__ __forceinline__ unsigned query(int row, int pos, int e) const {
        if (e >= a.dim + a.rot_dim) return 0;                      // dim and rot_dim are multiples of 8: pairs do not straddle
        const float* q = a.q + (size_t)row * a.ldq + h * (a.dim + a.rot_dim);
        const float qs = a.scale * 1.4426950408889634f;            // scores in units of log 2
        float u = q[e], v = q[e + 1];
        const int er = e - a.dim;
        if (er >= 0 && er < a.rot_dims) {
            const size_t at = (size_t)pos * (a.rot_dims / 2) + (er >> 1);
            const float c = a.rope_cos[at], s = a.rope_sin[at], x = u;
            u = fmaf(x, c, -(v * s));
            v = fmaf(v, c, x * s);
        }
        return pack_bf(u * qs, v * qs);
    }
    __device__ __forceinline__ int pieces() const { return (a.dim + a.rot_dim + a.vdim) / 8; }
    __device__ __forceinline__ FlashPiece piece(int v) const {
        const int kvec = a.dim / 8, rvec = a.rot_dim / 8;
        if (v < kvec) return {a.kv + h * a.dim + v * 8, a.ldkv, v, false};
        if (v < kvec + rvec) return {cache + a.rp + (v - kvec) * 8, a.ld, v, false};
        return {a.kv + a.heads * a.dim + h * a.vdim + (v - kvec - rvec) * 8, a.ldkv, v - kvec - rvec, true};
    }
    __device__ __forceinline__ float inverse(float m, float l) const {
        if (!a.sink) return 1.0f / l;
        const float s2 = a.sink[h] * 1.4426950408889634f, top = fmaxf(m, s2), e = exp2f(m - top);
        return e / (l * e + exp2f(s2 - top));
    }
    __device__ __forceinline__ void store(int row, int, int v, float o0, float o1) const {
        if (v >= a.vdim) return;
        const float* gate = a.y + (size_t)row * a.ldy + a.gate_off + h * a.vdim;
        bf16* out = static_cast<bf16*>(a.out) + (size_t)row * a.ldo + h * a.vdim;
        *reinterpret_cast<unsigned*>(out + v) = pack_bf(o0 * sigmoid_fast(gate[v]), o1 * sigmoid_fast(gate[v + 1]));
    }
};

// One head x 64 query rows; DV = value dimensions rounded up to a multiple of 64.
template <int DV>
__global__ void __launch_bounds__(FL_WARPS * 32, 2) k_latent_flash(const LatentArgs a) {
    flash_tile<DV>(LatentFlash(a, blockIdx.y), FlashShape{a.dim + a.rot_dim, a.window, a.cap, a.M}, a.seq);
}

// ------------------------------------------------------------------------------------------------------ host side
// Runs of at least 32 tokens of one sequence with bfloat16 activations and head sizes in whole 16-byte pieces.
static bool takes_flash(int M, bool one_seq, int dtype, int heads, int dim, int rot_dim, int vdim) {
    return one_seq && dtype == DET_BF16 && M >= 32 && !(float_flags() & 8) && dim % 8 == 0 && rot_dim % 8 == 0 && vdim % 8 == 0 &&
           vdim <= 256 && dim + rot_dim + vdim <= 768 && flash_smem(dim + rot_dim, (vdim + 63) / 64 * 64) <= 220 * 1024;
}
static int latent_rp(int kv_rank) { return round8(kv_rank); }

// Key ranges per row: enough CTAs to fill the device, at least 64 keys each.
static void plan_splits(int M, int heads, int window, int max_pos, int sms, int* splits, int* per_split) {
    const int keys = window > 0 ? std::min(window, max_pos + 1) : max_pos + 1;
    const long long ctas = (long long)M * ((heads + LS_WARPS - 1) / LS_WARPS);
    int s = (int)std::min<long long>((keys + 63) / 64, std::max<long long>(1, 3ll * sms / ctas));
    s = std::max(1, std::min(s, 256));
    *per_split = ((keys + s - 1) / s + LS_KEYS - 1) / LS_KEYS * LS_KEYS;
    *splits = (keys + *per_split - 1) / *per_split;
}

template <class T, int NP>
static void launch_scores(const LatentArgs& a, cudaStream_t q) {
    const size_t smem = 2 * LS_KEYS * 64 * NP * sizeof(T);
    static bool configured = false;
    if (!configured) {
        DETB_CUDA_OK(cudaFuncSetAttribute(k_latent_scores<T, NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        configured = true;
    }
    launch_pdl(k_latent_scores<T, NP>, dim3(a.splits, (a.heads + LS_WARPS - 1) / LS_WARPS, a.M), dim3(LS_WARPS * 32), smem, q, 1, a);
}
template <class T>
static void scores(const LatentArgs& a, cudaStream_t q) {
    const int np = (a.ld + 63) / 64;
    if (np <= 2) launch_scores<T, 2>(a, q);
    else if (np <= 5) launch_scores<T, 5>(a, q);
    else if (np <= 9) launch_scores<T, 9>(a, q);
    else if (np <= 17) launch_scores<T, 17>(a, q);
    else DETB_REQUIRE(false, "latent attention: the cached row is too wide");
}
template <int DV>
static void launch_flash(const LatentArgs& a, cudaStream_t q) {
    const size_t smem = flash_smem(a.dim + a.rot_dim, DV);
    static size_t configured = 0;
    if (smem > configured) {
        DETB_CUDA_OK(cudaFuncSetAttribute(k_latent_flash<DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        configured = smem;
    }
    launch_plain(k_latent_flash<DV>, dim3((a.M + FL_ROWS - 1) / FL_ROWS, a.heads), dim3(FL_WARPS * 32), smem, q, a);
}

static LatentArgs latent_args(const det_flatent_op* op) {
    DETB_REQUIRE(op->heads > 0 && op->dim > 0 && op->rot_dim >= 0 && op->vdim > 0 && op->q_rank > 0 && op->kv_rank > 0,
                 "latent attention: bad sizes");
    DETB_REQUIRE(op->rot_dims % 2 == 0 && op->rot_dims <= op->rot_dim && op->cap > 0, "latent attention: bad sizes");
    LatentArgs a{};
    a.heads = op->heads; a.dim = op->dim; a.rot_dim = op->rot_dim; a.rot_dims = op->rot_dims; a.vdim = op->vdim;
    a.q_rank = op->q_rank; a.kv_rank = op->kv_rank;
    a.rp = latent_rp(op->kv_rank);
    a.ld = det_f_latent_ld(op->kv_rank, op->rot_dim);
    a.window = op->window; a.scale = op->scale; a.cap = op->cap; a.M = op->M;
    a.y = op->y; a.ldy = op->ldy; a.dq_off = op->dq_off; a.dkv_off = op->dkv_off; a.gate_off = op->gate_off;
    a.dq_norm = op->dq_norm; a.dkv_norm = op->dkv_norm; a.eps = op->eps;
    a.rope_cos = op->rope_cos; a.rope_sin = op->rope_sin;
    a.cq = op->cq; a.ldcq = op->ldcq;
    a.q = op->q; a.ldq = op->ldq;
    a.sink = op->sink; a.out = op->out; a.ldo = op->ldo;
    a.seq = op->seq;
    return a;
}

}  // namespace detb

using namespace detb;

extern "C" {

int det_f_latent_ld(int kv_rank, int rot_dim) { return round8(kv_rank) + round8(rot_dim); }

size_t det_f_latent_scratch_bytes(int M, int heads, int dim, int rot_dim, int vdim, int kv_rank, int window, int cap, int max_pos,
                                  int dtype) {
    // the larger of the two forms; the split count grows as M shrinks, so a bound that holds for any M up to this one
    int splits = 1, per = 0;
    plan_splits(1, heads, window, max_pos, 148, &splits, &per);
    const size_t ld = (size_t)det_f_latent_ld(kv_rank, rot_dim);
    const size_t groups = (size_t)(heads + LS_WARPS - 1) / LS_WARPS;
    const size_t pieces = std::max<size_t>((size_t)M, std::min<size_t>((size_t)M * splits, 3 * 148 / std::max<size_t>(1, groups) + (size_t)M));
    const size_t absorbed = ((size_t)M * heads * ld + pieces * heads * (kv_rank + 2)) * sizeof(float);
    const size_t rows = (size_t)std::min(cap, max_pos + 1);
    const size_t expanded = dtype == DET_BF16 && M >= 32 ? rows * round8(heads * (dim + vdim)) * 2 : 0;
    return std::max(absorbed, expanded) + 256;
}

void det_f_latent_prep(const det_flatent_op* op, cudaStream_t st) {
    const LatentArgs a = latent_args(op);
    if (op->M <= 0) return;
    if (op->dtype == DET_BF16) launch_pdl(k_latent_prep<bf16>, dim3(op->M), dim3(256), 0, queue_of(st), 1, a);
    else launch_pdl(k_latent_prep<float>, dim3(op->M), dim3(256), 0, queue_of(st), 1, a);
}

void det_f_latent_attn(const det_flatent_op* op, cudaStream_t st) {
    LatentArgs a = latent_args(op);
    if (op->M <= 0) return;
    const det_flinear& w = *op->wkv;
    DETB_REQUIRE(w.N == op->heads * (op->dim + op->vdim) && w.K == op->kv_rank && w.ld == latent_rp(op->kv_rank),
                 "latent attention: the expansion weights do not fit");
    a.wkv = static_cast<const bf16*>(w.w);
    a.ldw = w.ld;
    cudaStream_t q = queue_of(st);
    const bool one = op->seq.table == nullptr;
    if (one && !op->seq.pos && takes_flash(op->M, one, op->dtype, op->heads, op->dim, op->rot_dim, op->vdim)) {
        const int rows = std::min(op->cap, op->seq.pos0 + op->M);
        bf16* kv = static_cast<bf16*>(op->scratch);
        det_fgemm_op g{};
        g.lin = &w;
        g.dtype = DET_BF16;
        g.x = op->seq.one.cache;
        g.ldx = a.ld;
        g.nseg = 1;
        g.seg_end[0] = w.N;
        g.glu_from = w.N;
        g.M = rows;
        g.y = kv;
        g.y_bf16 = 1;
        g.ldy = round8(w.N);
        det_f_gemm(&g, st);
        a.kv = kv;
        a.ldkv = round8(w.N);
        switch ((op->vdim + 63) / 64) {
            case 1: launch_flash<64>(a, q); break;
            case 2: launch_flash<128>(a, q); break;
            case 3: launch_flash<192>(a, q); break;
            default: launch_flash<256>(a, q); break;
        }
        return;
    }
    plan_splits(op->M, op->heads, op->window, op->max_pos, sm_count(), &a.splits, &a.per_split);
    a.qa = static_cast<float*>(op->scratch);
    a.part = a.qa + (size_t)op->M * op->heads * a.ld;
    const size_t absorb_smem = ((size_t)AB_ROWS * op->dim + 4 * AB_ROWS * AB_COLS) * sizeof(float);
    DETB_REQUIRE(absorb_smem <= 48 * 1024, "latent attention: the head is too large");
    launch_pdl(k_latent_absorb, dim3(op->heads, (a.rp + AB_COLS - 1) / AB_COLS, (op->M + AB_ROWS - 1) / AB_ROWS), dim3(128), absorb_smem,
               q, 1, a);
    if (op->dtype == DET_BF16) scores<bf16>(a, q);
    else scores<float>(a, q);
    const size_t smem = ((size_t)round8(op->kv_rank) + a.splits) * sizeof(float);
    dim3 grid(op->heads, (op->vdim + LO_V - 1) / LO_V, op->M);
    if (op->dtype == DET_BF16) launch_pdl(k_latent_out<bf16>, grid, dim3(256), smem, q, 1, a);
    else launch_pdl(k_latent_out<float>, grid, dim3(256), smem, q, 1, a);
}

}  // extern "C"
