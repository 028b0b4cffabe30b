// Products with fp32 activations (bfloat16 weights widened exactly, fp32 multiply-adds on the CUDA cores), the decay
// projection of the linear recurrences, and the entry that picks a kernel for det_f_gemm by shape.
#include "fops.cuh"
#include <algorithm>

namespace detb {

constexpr int SG_N = 64, SG_M = 64, SG_K = 16, SG_THREADS = 256;

struct DecayArgs {
    const bf16* w;
    int N, K, ldw;
    const float* low;
    int ldlow;
    const float* bias;
    int kind;
    float inv_tau;
    int M;
    float* z;
};

// One 64 (rows of W) x 64 (tokens) tile per CTA; thread (i, j) owns a 4 x 4 block.  acc[r][t]: weight row r, token t.
template <class LoadX>
__device__ __forceinline__ void simt_tile(const bf16* w, int ldw, int n0, int n_end, int K, int t0, int M, LoadX load_x,
                                          float (&acc)[4][4]) {
    __shared__ __align__(16) float ws[SG_K][SG_N + 4];
    __shared__ __align__(16) float xs[SG_K][SG_M + 4];
    const int tid = threadIdx.x, tr = tid & 15, tc = tid >> 4;
#pragma unroll
    for (int r = 0; r < 4; r++)
#pragma unroll
        for (int t = 0; t < 4; t++) acc[r][t] = 0.0f;
    for (int k0 = 0; k0 < K; k0 += SG_K) {
#pragma unroll
        for (int i = tid; i < SG_N * SG_K; i += SG_THREADS) {
            const int k = i & (SG_K - 1), n = i / SG_K;
            ws[k][n] = (n0 + n < n_end && k0 + k < K) ? to_f(w[(size_t)(n0 + n) * ldw + k0 + k]) : 0.0f;
            xs[k][n] = (t0 + n < M && k0 + k < K) ? load_x(t0 + n, k0 + k) : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < SG_K; k++) {
            const float4 a = *reinterpret_cast<const float4*>(&ws[k][tr * 4]);
            const float4 b = *reinterpret_cast<const float4*>(&xs[k][tc * 4]);
            const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int r = 0; r < 4; r++)
#pragma unroll
                for (int t = 0; t < 4; t++) acc[r][t] = fmaf(av[r], bv[t], acc[r][t]);
        }
        __syncthreads();
    }
}

__global__ void __launch_bounds__(SG_THREADS) k_fgemm_simt(const FgemmArgs a) {
    pdl_trigger();
    pdl_wait();
    TilePlace pl;
    int t0 = blockIdx.y * SG_M, t_end = a.M, n_base = 0;
    if (a.group_rows) {
        if ((int)blockIdx.y >= *a.nwork) return;
        const int4 w = a.work[blockIdx.y];
        n_base = w.x * a.group_rows;
        pl = TilePlace{0, n_base + (int)blockIdx.x * SG_N, n_base + a.group_rows};
        t0 = w.y;
        t_end = w.z;
    } else {
        pl = place_tile<SG_N>(a, blockIdx.x);
    }
    const float* x = static_cast<const float*>(a.x) + (size_t)a.seg_in[pl.seg] * a.gstride;
    float acc[4][4];
    simt_tile(a.w, a.ldw, pl.n0, pl.n_end, a.K, t0, t_end, [&](int t, int k) { return x[(size_t)t * a.ldx + k]; }, acc);
    const int tr = threadIdx.x & 15, tc = threadIdx.x >> 4;
#pragma unroll
    for (int t = 0; t < 4; t++) {
        const int m = t0 + tc * 4 + t;
        if (m >= t_end) continue;
        if (pl.n0 >= a.glu_from) {
            float* h = static_cast<float*>(a.h) + (size_t)m * a.ldh;
#pragma unroll
            for (int r = 0; r < 4; r++) {
                const int n = pl.n0 + tr * 4 + r;
                if (n >= pl.n_end) continue;
                if (a.act == DET_FF_RELU2) h[n - n_base - a.glu_from] = relu_squared(acc[r][t]);
                else if (!(r & 1)) h[(n - a.glu_from) / 2] = gate_pair(a.act, acc[r][t], acc[r | 1][t]);
            }
            continue;
        }
#pragma unroll
        for (int r = 0; r < 4; r++) {
            const int n = pl.n0 + tr * 4 + r;
            if (n >= pl.n_end) continue;
            float v = acc[r][t];
            if (a.bias) v += a.bias[n];
            if (a.softcap > 0.0f) v = a.softcap * tanhf(v / a.softcap);
            const size_t at = (size_t)m * a.ldy + n - n_base;
            if (a.yb) put(a.yb + at, v);
            else a.y[at] = a.accumulate ? a.y[at] + v : v;
        }
    }
}

__global__ void __launch_bounds__(SG_THREADS) k_fdecay(const DecayArgs a) {
    pdl_trigger();
    pdl_wait();
    const int n0 = blockIdx.x * SG_N, t0 = blockIdx.y * SG_M;
    float acc[4][4];
    simt_tile(a.w, a.ldw, n0, a.N, a.K, t0, a.M,
              [&](int t, int k) {
                  const float v = a.low[(size_t)t * a.ldlow + k];
                  return a.kind == DET_DECAY_EXP ? tanhf(v) : v;
              },
              acc);
    const int tr = threadIdx.x & 15, tc = threadIdx.x >> 4;
#pragma unroll
    for (int t = 0; t < 4; t++)
#pragma unroll
        for (int r = 0; r < 4; r++) {
            const int m = t0 + tc * 4 + t, n = n0 + tr * 4 + r;
            if (m < a.M && n < a.N) a.z[(size_t)m * a.N + n] = decay_of(acc[r][t] + a.bias[n], a.kind, a.inv_tau);
        }
}

void fgemm_simt_launch(FgemmArgs a, cudaStream_t q) {
    plan_tiles(a, SG_N);
    launch_pdl(k_fgemm_simt, dim3(a.tile0[a.nseg], (a.M + SG_M - 1) / SG_M), dim3(SG_THREADS), 0, q, 1, a);
}

// Token tiles of a work list: enough rows for what a linear of the stack gets on average.
int fgemm_group_tok(int dtype, int rows) {
    if (dtype != DET_BF16) return SG_M;
    return rows <= 24 ? 32 : 128;
}
void fgemm_group_launch(FgemmArgs a, int dtype, int tok, cudaStream_t q) {
    if (dtype == DET_BF16) {
        fgemm_tc_group_launch(a, tok, q);
        return;
    }
    launch_pdl(k_fgemm_simt, dim3((a.group_rows + SG_N - 1) / SG_N, a.max_work), dim3(SG_THREADS), 0, q, 1, a);
}

void fdecay_launch(const det_flinear* w2, const float* low, int ldlow, const float* bias, int kind, float tau, int M, float* z,
                   cudaStream_t q) {
    DecayArgs a;
    a.w = static_cast<const bf16*>(w2->w);
    a.N = w2->N; a.K = w2->K; a.ldw = w2->ld;
    a.low = low; a.ldlow = ldlow; a.bias = bias;
    a.kind = kind; a.inv_tau = 1.0f / tau;
    a.M = M; a.z = z;
    launch_pdl(k_fdecay, dim3((a.N + SG_N - 1) / SG_N, (M + SG_M - 1) / SG_M), dim3(SG_THREADS), 0, q, 1, a);
}

}  // namespace detb

using namespace detb;

extern "C" void det_f_gemm(const det_fgemm_op* op, cudaStream_t st) {
    const det_flinear& l = *op->lin;
    if (op->M <= 0) return;
    DETB_REQUIRE(l.N > 0 && l.K > 0 && l.ld % 8 == 0 && l.ld >= l.K && (reinterpret_cast<uintptr_t>(l.w) & 15) == 0,
                 "linear: bad layout");
    DETB_REQUIRE(op->ldx % 8 == 0 && op->ldx >= l.ld && (reinterpret_cast<uintptr_t>(op->x) & 15) == 0 && op->group_stride % 8 == 0,
                 "linear: bad input layout");
    DETB_REQUIRE(op->nseg >= 1 && op->nseg <= 8 && op->seg_end[op->nseg - 1] == l.N, "linear: bad segments");
    FgemmArgs a{};
    a.w = static_cast<const bf16*>(l.w);
    a.wt = static_cast<const bf16*>(l.wt);
    a.N = l.N; a.K = l.K; a.ldw = l.ld;
    a.x = op->x; a.ldx = op->ldx; a.gstride = op->group_stride;
    a.nseg = op->nseg;
    bool glu_ok = op->glu_from >= l.N;
    for (int i = 0, start = 0; i < op->nseg; i++) {
        a.seg_end[i] = op->seg_end[i];
        a.seg_in[i] = op->seg_in[i];
        DETB_REQUIRE(op->seg_end[i] > start && op->seg_in[i] >= 0, "linear: bad segments");
        DETB_REQUIRE(!op->norm_x || op->seg_in[i] == 0, "linear: a normalised input has one group");
        glu_ok = glu_ok || start == op->glu_from;
        DETB_REQUIRE(start < op->glu_from || op->act == DET_FF_RELU2 || (op->seg_end[i] - start) % 2 == 0, "linear: an odd number of pair rows");
        start = op->seg_end[i];
    }
    DETB_REQUIRE(glu_ok, "linear: the pair rows must start a segment");
    DETB_REQUIRE(op->glu_from == 0 || op->y, "linear: no output");
    DETB_REQUIRE(op->glu_from >= l.N || op->h, "linear: no pair output");
    a.glu_from = op->glu_from;
    a.M = op->M;
    a.y = op->y_bf16 ? nullptr : static_cast<float*>(op->y);
    a.yb = op->y_bf16 ? static_cast<bf16*>(op->y) : nullptr;
    DETB_REQUIRE(!(op->y_bf16 && op->accumulate), "linear: bfloat16 outputs do not accumulate");
    a.ldy = op->ldy;
    a.accumulate = op->accumulate;
    a.softcap = op->softcap;
    a.h = op->h; a.ldh = op->ldh;
    a.bias = op->bias;
    a.act = op->act;
    DETB_REQUIRE(op->act >= DET_FF_SWIGLU && op->act <= DET_FF_RELU2, "linear: unknown activation");
    a.error_flag = error_word();
    cudaStream_t q = queue_of(st);
    if (op->norm_x) {
        a.norm_x = op->norm_x; a.norm_w = op->norm_w; a.eps = op->eps;
        if ((float_flags() & 1) || !fgemv_takes(a, op->dtype)) {
            det_fnorm_op n{};
            n.x = op->norm_x; n.w = op->norm_w; n.eps = op->eps;
            n.M = op->M; n.n = l.K; n.dtype = op->dtype;
            n.out = const_cast<void*>(op->x); n.ld = op->ldx;
            det_f_norm(&n, st);
            a.norm_x = nullptr;
        }
    }
    if (fgemv_takes(a, op->dtype)) fgemv_launch(a, op->dtype, q);
    else if (op->dtype == DET_BF16) fgemm_tc_launch(a, q);
    else fgemm_simt_launch(a, q);
}
