// RMS norm of residual rows for the floating-point op set, with the token-shift mixes of a recurrent mixer in the same
// launch: out group g = h + (h' - h) * mu[g], the last group = h.  One block per row.  The row before comes from the same
// residual rows (its norm is recomputed: one more read of a row that is in L2) or, for the first token of a step, from the
// sequence's state; both are fp32, so a mix does not depend on where a step was cut.
#include "fops.cuh"
#include <algorithm>

namespace detb {

constexpr int NORM_THREADS = 256;

// 1 / sqrt(mean(x^2) + eps) of a row (16-byte loads when the row allows them)
__device__ __forceinline__ float row_rstd(const float* __restrict__ x, int n, float eps, float* sh) {
    float s = 0.0f;
    if ((n & 3) == 0 && (reinterpret_cast<uintptr_t>(x) & 15) == 0) {
        for (int i = threadIdx.x; i < n / 4; i += NORM_THREADS) {
            const float4 v = reinterpret_cast<const float4*>(x)[i];
            s = fmaf(v.x, v.x, s);
            s = fmaf(v.y, v.y, s);
            s = fmaf(v.z, v.z, s);
            s = fmaf(v.w, v.w, s);
        }
    } else {
        for (int i = threadIdx.x; i < n; i += NORM_THREADS) s = fmaf(x[i], x[i], s);
    }
    return 1.0f / sqrtf(block_sum(s, sh) / (float)n + eps);
}
template <int V>
__device__ __forceinline__ void load_v(const float* p, float (&v)[V]) {
    if constexpr (V == 4) {
        const float4 f = *reinterpret_cast<const float4*>(p);
        v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
    } else {
        v[0] = *p;
    }
}
template <int V>
__device__ __forceinline__ void store_v(float* p, const float (&v)[V]) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else *p = v[0];
}
template <int V>
__device__ __forceinline__ void store_v(bf16* p, const float (&v)[V]) {
    if constexpr (V == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf(v[0], v[1]), pack_bf(v[2], v[3]));
    else put(p, v[0]);
}

// grid (rows, column pieces): every block of a row takes the row's sum of squares itself and writes its columns.
// V columns per thread and pass: 4, or 1 for row lengths that are not a multiple of 4.
template <class T, int V>
__global__ void __launch_bounds__(NORM_THREADS) k_fnorm(const det_fnorm_op a) {
    __shared__ float sh[32];
    pdl_trigger();
    pdl_wait();
    const int r = blockIdx.x;
    const float* x = a.x + (size_t)(a.rows ? a.rows[r] : r) * a.n;
    T* out = static_cast<T*>(a.out) + (size_t)r * a.ld;
    const int per = ((a.n + V - 1) / V + gridDim.y - 1) / gridDim.y * V;      // columns of a piece
    const int c0 = blockIdx.y * per, c1 = min(a.n, c0 + per);
    const float rs = row_rstd(x, a.n, a.eps, sh);
    if (a.nmix == 0) {
        for (int i = c0 + threadIdx.x * V; i < c1; i += NORM_THREADS * V) {
            float v[V], w[V];
            load_v(x + i, v);
            load_v(a.w + i, w);
#pragma unroll
            for (int j = 0; j < V; j++) v[j] = v[j] * rs * w[j];
            store_v(out + i, v);
        }
        return;
    }
    const bool own = a.seq.table != nullptr;          // every row is its own sequence
    const bool from_state = own || r == 0;
    const float* xp = x - a.n;
    float rp = 0.0f, rl = 0.0f;
    const float* xl = a.x + (size_t)(own ? r : a.M - 1) * a.n;
    if (!from_state) rp = row_rstd(xp, a.n, a.eps, sh);
    else rl = xl == x ? rs : row_rstd(xl, a.n, a.eps, sh);
    float* prev = from_state ? slot_of(a.seq, r).prev : nullptr;
    for (int i = c0 + threadIdx.x * V; i < c1; i += NORM_THREADS * V) {
        float w[V], h[V], d[V];
        load_v(a.w + i, w);
        load_v(x + i, h);
        if (from_state) {
            float last[V];
            load_v(prev + i, d);
            load_v(xl + i, last);
#pragma unroll
            for (int j = 0; j < V; j++) last[j] = last[j] * rl * w[j];
            store_v(prev + i, last);                  // this thread has read these columns; no other touches them
        } else {
            load_v(xp + i, d);
#pragma unroll
            for (int j = 0; j < V; j++) d[j] = d[j] * rp * w[j];
        }
#pragma unroll
        for (int j = 0; j < V; j++) {
            h[j] = h[j] * rs * w[j];
            d[j] -= h[j];
        }
        for (int g = 0; g < a.nmix; g++) {
            float mu[V], y[V];
            load_v(a.mu + (size_t)g * a.n + i, mu);
#pragma unroll
            for (int j = 0; j < V; j++) y[j] = fmaf(d[j], mu[j], h[j]);
            store_v(out + g * a.group_stride + i, y);
        }
        store_v(out + a.nmix * a.group_stride + i, h);
    }
}

template <class T>
static void launch_norm(const det_fnorm_op& op, cudaStream_t q) {
    // few rows: cut them into pieces of at least 256 columns, so that a decoded token is not one block's work
    const int pieces = std::max(1, std::min(2 * sm_count() / op.M, (op.n + 255) / 256));
    const dim3 grid(op.M, op.nmix ? pieces : std::min(pieces, 4));
    if (op.n % 4 == 0) launch_pdl(k_fnorm<T, 4>, grid, dim3(NORM_THREADS), 0, q, 1, op);
    else launch_pdl(k_fnorm<T, 1>, grid, dim3(NORM_THREADS), 0, q, 1, op);
}

}  // namespace detb

using namespace detb;

static int g_float_flags = 0;
int detb::float_flags() { return g_float_flags; }

extern "C" {

void det_debug_set_float(int flags) { g_float_flags = flags; }

void det_f_norm(const det_fnorm_op* op, cudaStream_t st) {
    DETB_REQUIRE(op->n > 0 && op->ld % 8 == 0 && op->ld >= op->n && (op->nmix == 0 || !op->rows), "norm: bad shape");
    if (op->M <= 0) return;
    auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    DETB_REQUIRE(aligned(op->out) && op->group_stride % 8 == 0 && (op->n % 4 != 0 || (aligned(op->x) && aligned(op->w) && aligned(op->mu))),
                 "norm: rows must be 16-byte aligned");
    if (op->dtype == DET_BF16) launch_norm<bf16>(*op, queue_of(st));
    else launch_norm<float>(*op, queue_of(st));
}

}  // extern "C"
