// Pieces shared by the floating-point op set (include/det_b200.h, Part 3): activation element access, warp and block sums,
// which sequence and position a row belongs to.  Unlike the quantized ops these kernels carry no bit-for-bit contract;
// sums use fused multiply-adds in a fixed order, so a launch of the same shape always gives the same bits.
#pragma once
#include "gemm_common.cuh"
#include <cuda_bf16.h>

namespace detb {

using bf16 = __nv_bfloat16;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(bf16* p, float v) { *p = __float2bfloat16_rn(v); }
// the two bfloat16 values of a 32-bit word, lower address first
__device__ __forceinline__ float bf_lo(unsigned w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float bf_hi(unsigned w) { return __uint_as_float(w & 0xffff0000u); }
__device__ __forceinline__ unsigned pack_bf(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const unsigned*>(&v);
}

__device__ __forceinline__ float sigmoid_fast(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu_fast(float z) { return z / (1.0f + expf(-z)); }
// first half of a feed-forward (DET_FF_*)
__device__ __forceinline__ float gate_pair(int act, float g, float u) { return (act == DET_FF_REGLU ? fmaxf(g, 0.0f) : silu_fast(g)) * u; }
__device__ __forceinline__ float relu_squared(float v) {
    const float r = fmaxf(v, 0.0f);
    return r * r;
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) v += __shfl_xor_sync(FULL, v, off);
    return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) v = fmaxf(v, __shfl_xor_sync(FULL, v, off));
    return v;
}
// Sum over the block (blockDim.x a multiple of 32); `sh` holds 32 floats.  Every thread gets the total.
__device__ __forceinline__ float block_sum(float v, float* sh) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    v = warp_sum(v);
    __syncthreads();
    if (lane == 0) sh[warp] = v;
    __syncthreads();
    return warp_sum(lane < nw ? sh[lane] : 0.0f);
}

__device__ __forceinline__ det_seq_slot slot_of(const det_seq_ref& r, int row) { return r.table ? r.table[row] : r.one; }
__device__ __forceinline__ int position_of(const det_seq_ref& r, int row) {
    if (r.table) return r.pos[row];
    return (r.pos ? *r.pos : r.pos0) + row;
}

// ---- entries between the translation units
struct FgemmArgs {
    const bf16* w;
    const bf16* wt;          // tile-major copy, or NULL
    int N, K, ldw;
    const void* x;
    int ldx;
    long long gstride;
    int nseg;
    int seg_end[8], seg_in[8];
    int tile0[9];            // first tile of each segment (tiles of the launched kernel's row count), [nseg] = total
    int glu_from;
    int M;
    const float* norm_x;     // GEMV prologue only
    const float* norm_w;
    float eps;
    float* y;
    bf16* yb;                // bfloat16 output instead of y
    int ldy;
    int accumulate;
    float softcap;
    void* h;
    int ldh;
    const float* bias;       // of rows before glu_from, or NULL
    int act;
    int* error_flag;
    // Stacked linears (one per expert, group_rows rows each): which rows meet which linear is known on the device only.
    int group_rows;          // 0: one linear
    const int* sel;          // GEMV: linear of pair p, whose input is row p / pairs_per_row; >= groups: none
    int groups, pairs, pairs_per_row;
    const int4* work;        // GEMM: {linear, first row, row after the last, -} per token tile
    const int* nwork;
    int max_work;
};
// Segment of tile `t` and the first weight row of the tile (tiles of ROWS rows never straddle a segment).
struct TilePlace {
    int seg, n0, n_end;
};
template <int ROWS>
__device__ __forceinline__ TilePlace place_tile(const FgemmArgs& a, int t) {
    int s = 0;
#pragma unroll
    for (int j = 1; j < 8; j++)
        if (j < a.nseg && t >= a.tile0[j]) s = j;
    const int start = s ? a.seg_end[s - 1] : 0;
    return TilePlace{s, start + (t - a.tile0[s]) * ROWS, a.seg_end[s]};
}
inline void plan_tiles(FgemmArgs& a, int rows) {
    int t = 0, start = 0;
    for (int s = 0; s < a.nseg; s++) {
        a.tile0[s] = t;
        t += (a.seg_end[s] - start + rows - 1) / rows;
        start = a.seg_end[s];
    }
    for (int s = a.nseg; s < 9; s++) a.tile0[s] = t;
}
inline int round8(int n) { return (n + 7) & ~7; }

bool fgemv_takes(const FgemmArgs& a, int dtype);                         // fgemv.cu
void fgemv_launch(FgemmArgs a, int dtype, cudaStream_t q);
void fgemm_tc_launch(FgemmArgs a, cudaStream_t q);                       // fgemm_tc.cu (bfloat16 activations)
void fgemm_simt_launch(FgemmArgs a, cudaStream_t q);                     // fgemm.cu (fp32 activations)
// The same over stacked linears; `a` carries group_rows and sel (GEMV) or work (GEMM).  Tiles of a work list have
// fgemm_group_tok(dtype, rows per linear) tokens.
bool fgemv_group_takes(const FgemmArgs& a, int rows);
void fgemv_group_launch(FgemmArgs a, int dtype, cudaStream_t q);
int fgemm_group_tok(int dtype, int rows);
void fgemm_group_launch(FgemmArgs a, int dtype, int tok, cudaStream_t q);
void fgemm_tc_group_launch(FgemmArgs a, int tok, cudaStream_t q);
// z[M][N] = f(W act(x) + bias), all in 32-bit (the decay of a linear recurrence)
void fdecay_launch(const det_flinear* w2, const float* low, int ldlow, const float* bias, int kind, float tau, int M, float* z,
                   cudaStream_t q);
int float_flags();

// decay of a key channel from its projection
__device__ __forceinline__ float decay_of(float z, int kind, float inv_tau) {
    if (kind == DET_DECAY_SIGMOID) {
        // log sigmoid(z) = min(z, 0) - log1p(exp(-|z|))
        const float ls = fminf(z, 0.0f) - log1pf(expf(-fabsf(z)));
        return expf(ls * inv_tau);
    }
    return expf(-expf(z));
}

}  // namespace detb
