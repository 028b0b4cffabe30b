// Minimal gated recurrence (include/det_b200.h, det_fmingru_op): per channel S <- (1 - z) S + z * candidate, a linear recurrence
// whose coefficients read only the current token.
//
//   k_fmingru_step   one token per row (decode, batches): elementwise.
//   k_fmingru_scan   a run of tokens: a CTA takes 32 channels, its warps consecutive pieces of SCAN_T tokens.  A warp reduces its
//                    piece to (product of 1 - z, state from zero), the pieces' entry states follow from those in order, and
//                    the warp replays its piece from registers: one read of the inputs, SCAN_WARPS * SCAN_T tokens per round.
// Bound by the bytes of the fp32 rows.
#include "fops.cuh"
#include <algorithm>

namespace detb {

__device__ __forceinline__ float mingru_candidate(float u) { return u >= 0.0f ? u + 0.5f : sigmoid_fast(u); }

template <class T>
__global__ void __launch_bounds__(256) k_fmingru_step(const det_fmingru_op a) {
    pdl_trigger();
    pdl_wait();
    const int i = blockIdx.x * 256 + threadIdx.x, row = blockIdx.y;
    if (i >= a.n) return;
    const float* y = a.y + (size_t)row * a.ldy;
    float* s = slot_of(a.seq, row).s + i;
    const float z = sigmoid_fast(y[a.z_off + i]);
    const float v = fmaf(z, mingru_candidate(y[a.x_off + i]), (1.0f - z) * *s);
    *s = v;
    put(static_cast<T*>(a.out) + (size_t)row * a.ldo + i, v * silu_fast(y[a.gate_off + i]));
}

constexpr int SCAN_T = 8, SCAN_WARPS = 16;      // 512 threads: three CTAs an SM

template <class T>
__global__ void __launch_bounds__(SCAN_WARPS * 32) k_fmingru_scan(const det_fmingru_op a) {
    __shared__ float prod[SCAN_WARPS][32], part[SCAN_WARPS][32], carry[32];
    pdl_trigger();
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    const int i = blockIdx.x * 32 + lane;
    const bool live = i < a.n;
    float* state = a.seq.one.s + i;
    if (warp == 0) carry[lane] = live ? *state : 0.0f;
    for (int base = 0; base < a.M; base += warps * SCAN_T) {
        const int t0 = base + warp * SCAN_T, nt = min(SCAN_T, a.M - t0);
        float keep[SCAN_T], add[SCAN_T], gate[SCAN_T];
#pragma unroll
        for (int t = 0; t < SCAN_T; t++) {
            keep[t] = 1.0f;
            add[t] = gate[t] = 0.0f;
            if (live && t < nt) {
                const float* y = a.y + (size_t)(t0 + t) * a.ldy + i;
                keep[t] = y[a.z_off];
                add[t] = y[a.x_off];
                gate[t] = y[a.gate_off];
            }
        }
        float p = 1.0f, s = 0.0f;
#pragma unroll
        for (int t = 0; t < SCAN_T; t++)
            if (live && t < nt) {
                const float z = sigmoid_fast(keep[t]);
                keep[t] = 1.0f - z;
                add[t] = z * mingru_candidate(add[t]);
                p *= keep[t];
                s = fmaf(keep[t], s, add[t]);
            }
        prod[warp][lane] = p;
        part[warp][lane] = s;
        __syncthreads();
        float in = carry[lane];
        for (int w = 0; w < warp; w++) in = fmaf(prod[w][lane], in, part[w][lane]);
#pragma unroll
        for (int t = 0; t < SCAN_T; t++)
            if (live && t < nt) {
                in = fmaf(keep[t], in, add[t]);
                put(static_cast<T*>(a.out) + (size_t)(t0 + t) * a.ldo + i, in * silu_fast(gate[t]));
            }
        __syncthreads();                      // every warp has read the carry and the pieces
        if (warp == warps - 1) carry[lane] = in;
        __syncthreads();
    }
    if (warp == 0 && live) *state = carry[lane];
}

}  // namespace detb

using namespace detb;

extern "C" void det_f_mingru(const det_fmingru_op* op, cudaStream_t st) {
    DETB_REQUIRE(op->n > 0 && op->ldo >= op->n, "gated recurrence: bad sizes");
    if (op->M <= 0) return;
    cudaStream_t q = queue_of(st);
    const bool bf = op->dtype == DET_BF16;
    if (op->seq.table || op->M == 1) {
        const dim3 grid((op->n + 255) / 256, op->M);
        if (bf) launch_pdl(k_fmingru_step<bf16>, grid, dim3(256), 0, q, 1, *op);
        else launch_pdl(k_fmingru_step<float>, grid, dim3(256), 0, q, 1, *op);
        return;
    }
    const int warps = std::min(SCAN_WARPS, (op->M + SCAN_T - 1) / SCAN_T);
    const dim3 grid((op->n + 31) / 32), block(warps * 32);
    if (bf) launch_pdl(k_fmingru_scan<bf16>, grid, block, 0, q, 1, *op);
    else launch_pdl(k_fmingru_scan<float>, grid, block, 0, q, 1, *op);
}
