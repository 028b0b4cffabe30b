// RMS norm of residual rows for the floating-point op set, with the token-shift mixes of a recurrent mixer in the same
// launch: out group g = h + (h' - h) * mu[g], the last group = h.  One block per row.  The row before comes from the same
// residual rows (its norm is recomputed: one more read of a row that is in L2) or, for the first token of a step, from the
// sequence's state; both are fp32, so a mix does not depend on where a step was cut.
#include "fops.cuh"

namespace detb {

constexpr int NORM_THREADS = 256;

__device__ __forceinline__ float row_rstd(const float* __restrict__ x, int n, float eps, float* sh) {
    float s = 0.0f;
    for (int i = threadIdx.x; i < n; i += NORM_THREADS) s = fmaf(x[i], x[i], s);
    return 1.0f / sqrtf(block_sum(s, sh) / (float)n + eps);
}

template <class T>
__global__ void __launch_bounds__(NORM_THREADS) k_fnorm(const det_fnorm_op a) {
    __shared__ float sh[32];
    pdl_trigger();
    pdl_wait();
    const int r = blockIdx.x;
    const float* x = a.x + (size_t)(a.rows ? a.rows[r] : r) * a.n;
    T* out = static_cast<T*>(a.out) + (size_t)r * a.ld;
    const float rs = row_rstd(x, a.n, a.eps, sh);
    if (a.nmix == 0) {
        for (int i = threadIdx.x; i < a.n; i += NORM_THREADS) put(out + i, x[i] * rs * a.w[i]);
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
    for (int i = threadIdx.x; i < a.n; i += NORM_THREADS) {
        const float w = a.w[i], h = x[i] * rs * w;
        float hp;
        if (from_state) {
            hp = prev[i];
            prev[i] = xl[i] * rl * w;                 // this thread has read prev[i]; no other block touches it
        } else {
            hp = xp[i] * rp * w;
        }
        for (int g = 0; g < a.nmix; g++) put(out + g * a.group_stride + i, fmaf(hp - h, a.mu[(size_t)g * a.n + i], h));
        put(out + a.nmix * a.group_stride + i, h);
    }
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
    if (op->dtype == DET_BF16) launch_pdl(k_fnorm<bf16>, dim3(op->M), dim3(NORM_THREADS), 0, queue_of(st), 1, *op);
    else launch_pdl(k_fnorm<float>, dim3(op->M), dim3(NORM_THREADS), 0, queue_of(st), 1, *op);
}

}  // extern "C"
