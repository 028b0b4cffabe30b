// Decode GEMV over bfloat16 weights: y[m][n] = sum_k W[n][k] x[m][k] for up to four rows m, fp32 products and sums.
//
// Bound by the bytes of W.  Persistent CTAs of sixteen warps; the input rows are staged once per CTA in shared memory as
// fp32 (RMS norm included when the call carries one), in two planes of four so that a lane's eight values are two
// conflict-free 16-byte loads.  A warp takes four weight rows ("quad") and a share of K: WSPLIT of a CTA's warps split K of
// one quad and add up through shared memory, chosen by shape so that the quads divide over the SMs without a ragged last
// round.  A lane holds eight 16-byte weight loads in flight; the first of them are issued before griddepcontrol.wait, since
// weights do not depend on the previous kernel.
#include "fops.cuh"
#include <algorithm>

namespace detb {

constexpr int GV_WARPS = 16, GV_THREADS = GV_WARPS * 32, GV_ROWS = 4;

struct GemvPlan {
    int wsplit;
    int kp;         // K rounded up to 8: elements of a staged row
    int ngroups;    // input groups staged
};

template <int R>
__device__ __forceinline__ void load_quad(const bf16* const (&row)[R], int k, int kp, uint4 (&w)[R]) {
#pragma unroll
    for (int r = 0; r < R; r++) w[r] = k < kp ? __ldcs(reinterpret_cast<const uint4*>(row[r] + k)) : make_uint4(0, 0, 0, 0);
}

// GROUPED: a quad belongs to a pair (input row, linear of a stack), chosen on the device; xs then holds every input row.
template <class T, int MT, bool NORM, bool GROUPED = false>
__global__ void __launch_bounds__(GV_THREADS, 1) k_fgemv(const FgemmArgs a, const GemvPlan p) {
    extern __shared__ __align__(16) float xs[];                     // [ngroups][MT][2 planes][kp / 2]
    __shared__ float red[2][GV_WARPS][GV_ROWS * MT];
    __shared__ float sh[32];
    pdl_trigger();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int ws = p.wsplit, group = warp / ws, part = warp % ws, qpc = GV_WARPS / ws;   // quads per CTA and round
    const int qpg = GROUPED ? (a.group_rows + GV_ROWS - 1) / GV_ROWS : 0;      // quads of a pair
    const int nquads = GROUPED ? a.pairs * qpg : a.tile0[a.nseg];
    const int kp = p.kp, half = kp / 2;
    const int stride = qpc * gridDim.x;
    int quad = blockIdx.x * qpc + group;

    const bf16* row[GV_ROWS];
    uint4 w0[GV_ROWS];
    TilePlace pl{};
    int pair = 0, n_base = 0;
    bool none = false;
    auto aim = [&](int t) {
        if constexpr (GROUPED) {
            pair = t / qpg;
            const int e = a.sel[pair];
            none = e >= a.groups;
            n_base = (none ? 0 : e) * a.group_rows;
            pl = TilePlace{pair / a.pairs_per_row, n_base + (t - pair * qpg) * GV_ROWS, n_base + a.group_rows};
        } else {
            pl = place_tile<GV_ROWS>(a, t);
        }
#pragma unroll
        for (int r = 0; r < GV_ROWS; r++) row[r] = a.w + (size_t)min(pl.n0 + r, pl.n_end - 1) * a.ldw;
    };
    const int kstep = ws * 256, k_first = (part * 32 + lane) * 8;
    if (!GROUPED && quad < nquads) {
        aim(quad);
        load_quad(row, k_first, kp, w0);
    }
    pdl_wait();
    if (GROUPED && quad < nquads) {
        aim(quad);
        if (!none) load_quad(row, k_first, kp, w0);
    }

    // ---- stage the input rows
    if constexpr (NORM) {
        for (int m = 0; m < a.M; m++) {
            const float* x = a.norm_x + (size_t)m * a.K;
            float s = 0.0f;
            for (int i = threadIdx.x; i < a.K; i += GV_THREADS) s = fmaf(x[i], x[i], s);
            const float rs = 1.0f / sqrtf(block_sum(s, sh) / (float)a.K + a.eps);
            float* dst = xs + (size_t)m * kp;
            for (int i = threadIdx.x; i < kp; i += GV_THREADS)
                dst[((i >> 2) & 1) * half + (i >> 3) * 4 + (i & 3)] = i < a.K ? x[i] * rs * a.norm_w[i] : 0.0f;
        }
    } else {
        for (int gm = 0; gm < p.ngroups * a.M; gm++) {
            const int g = gm / a.M, m = gm % a.M;
            const T* x = static_cast<const T*>(a.x) + g * a.gstride + (size_t)m * a.ldx;
            float* dst = xs + (size_t)(g * MT + m) * kp;
            for (int i = threadIdx.x; i < kp / 4; i += GV_THREADS) {
                float4 v;
                if constexpr (sizeof(T) == 2) {
                    const uint2 b = reinterpret_cast<const uint2*>(x)[i];
                    v = make_float4(bf_lo(b.x), bf_hi(b.x), bf_lo(b.y), bf_hi(b.y));
                } else {
                    v = reinterpret_cast<const float4*>(x)[i];
                }
                *reinterpret_cast<float4*>(dst + (i & 1) * half + (i >> 1) * 4) = v;
            }
        }
    }
    __syncthreads();

    int buf = 0;
    for (int base = blockIdx.x * qpc; base < nquads; base += stride, quad += stride, buf ^= 1) {
        const bool live = quad < nquads && !none;
        if (live) {
            const float* xg = xs + (size_t)(GROUPED ? pl.seg : a.seg_in[pl.seg]) * MT * kp;
            float acc[GV_ROWS][MT];
#pragma unroll
            for (int r = 0; r < GV_ROWS; r++)
#pragma unroll
                for (int m = 0; m < MT; m++) acc[r][m] = 0.0f;
            for (int k = k_first; k < kp; k += kstep) {
                uint4 w1[GV_ROWS];
                load_quad(row, k + kstep, kp, w1);
#pragma unroll
                for (int m = 0; m < MT; m++) {
                    const float4 xa = *reinterpret_cast<const float4*>(xg + m * kp + (k >> 1));
                    const float4 xb = *reinterpret_cast<const float4*>(xg + m * kp + half + (k >> 1));
#pragma unroll
                    for (int r = 0; r < GV_ROWS; r++) {
                        float s = acc[r][m];
                        s = fmaf(bf_lo(w0[r].x), xa.x, s);
                        s = fmaf(bf_hi(w0[r].x), xa.y, s);
                        s = fmaf(bf_lo(w0[r].y), xa.z, s);
                        s = fmaf(bf_hi(w0[r].y), xa.w, s);
                        s = fmaf(bf_lo(w0[r].z), xb.x, s);
                        s = fmaf(bf_hi(w0[r].z), xb.y, s);
                        s = fmaf(bf_lo(w0[r].w), xb.z, s);
                        s = fmaf(bf_hi(w0[r].w), xb.w, s);
                        acc[r][m] = s;
                    }
                }
#pragma unroll
                for (int r = 0; r < GV_ROWS; r++) w0[r] = w1[r];
            }
#pragma unroll
            for (int r = 0; r < GV_ROWS; r++)
#pragma unroll
                for (int m = 0; m < MT; m++) {
                    const float s = warp_sum(acc[r][m]);
                    if (lane == 0) red[buf][warp][r * MT + m] = s;
                }
        }
        const TilePlace here = pl;
        const int here_pair = pair, here_base = n_base;
        // the next quad's first weights are requested before this one is handed over
        if (quad + stride < nquads) {
            aim(quad + stride);
            if (!none) load_quad(row, k_first, kp, w0);
        }
        if (ws == 1) __syncwarp();
        else if (ws == GV_WARPS) __syncthreads();
        else asm volatile("bar.sync %0, %1;" ::"r"(1 + group), "r"(ws * 32) : "memory");
        if (live && part == 0 && lane < GV_ROWS * MT) {
            const int r = lane / MT, m = lane % MT, n = here.n0 + r;
            float v = 0.0f;
            for (int i = 0; i < ws; i++) v += red[buf][group * ws + i][lane];
            constexpr unsigned LANES = (1u << (GV_ROWS * MT)) - 1u;
            const float other = __shfl_down_sync(LANES, v, MT);     // row r + 1 of the quad, same m
            if (m < a.M && n < here.n_end) {
                if (n >= a.glu_from) {
                    if (a.act == DET_FF_RELU2)
                        put(static_cast<T*>(a.h) + (size_t)(GROUPED ? here_pair : m) * a.ldh + (n - here_base - a.glu_from), relu_squared(v));
                    else if (!(r & 1))
                        put(static_cast<T*>(a.h) + (size_t)m * a.ldh + (n - a.glu_from) / 2, gate_pair(a.act, v, other));
                } else {
                    if (a.bias) v += a.bias[n];
                    if (a.softcap > 0.0f) v = a.softcap * tanhf(v / a.softcap);
                    const size_t at = (size_t)m * a.ldy + n;
                    if (a.yb) put(a.yb + at, v);
                    else a.y[at] = a.accumulate ? a.y[at] + v : v;
                }
            }
        }
    }
}

static size_t gemv_smem(const FgemmArgs& a, int mt) {
    int groups = 1;
    for (int s = 0; s < a.nseg; s++) groups = std::max(groups, a.seg_in[s] + 1);
    return (size_t)groups * mt * round8(a.K) * sizeof(float);
}
static int gemv_mt(int m) { return m <= 1 ? 1 : (m <= 2 ? 2 : 4); }

bool fgemv_takes(const FgemmArgs& a, int) {
    if (float_flags() & 2) return false;
    return a.M <= 4 && gemv_smem(a, gemv_mt(a.M)) <= smem_optin() - 8192;
}

template <class T, int MT, bool NORM, bool GROUPED = false>
static void launch_gemv(const FgemmArgs& a, cudaStream_t q) {
    const size_t smem = gemv_smem(a, MT);
    static size_t configured = 0;
    if (smem > configured) {
        DETB_CUDA_OK(cudaFuncSetAttribute(k_fgemv<T, MT, NORM, GROUPED>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        configured = smem;
    }
    GemvPlan p;
    p.kp = round8(a.K);
    p.ngroups = (int)(smem / ((size_t)MT * p.kp * sizeof(float)));
    // warps per quad: the smallest split whose last round wastes little; a warp keeps at least one full step of K
    const int quads = GROUPED ? a.pairs * ((a.group_rows + GV_ROWS - 1) / GV_ROWS) : a.tile0[a.nseg], sms = sm_count();
    p.wsplit = 1;
    double best = 1e30;
    for (int ws = 1; ws <= GV_WARPS; ws *= 2) {
        if (ws > 1 && (ws - 1) * 256 >= p.kp) break;
        const int per_round = sms * (GV_WARPS / ws);
        const double cost = (double)((quads + per_round - 1) / per_round) * (1.0 / ws) * (1.0 + 0.02 * ws);
        if (cost < best * 0.999) {
            best = cost;
            p.wsplit = ws;
        }
    }
    const int qpc = GV_WARPS / p.wsplit;
    const int grid = std::min(sms, (quads + qpc - 1) / qpc);
    launch_pdl(k_fgemv<T, MT, NORM, GROUPED>, dim3(grid), dim3(GV_THREADS), smem, q, 1, a, p);
}

template <class T, int MT>
static void launch_norm(const FgemmArgs& a, cudaStream_t q) {
    if (a.norm_x) launch_gemv<T, MT, true>(a, q);
    else launch_gemv<T, MT, false>(a, q);
}
template <class T>
static void launch_mt(const FgemmArgs& a, cudaStream_t q) {
    switch (gemv_mt(a.M)) {
        case 1: launch_norm<T, 1>(a, q); break;
        case 2: launch_norm<T, 2>(a, q); break;
        default: launch_norm<T, 4>(a, q); break;
    }
}
void fgemv_launch(FgemmArgs a, int dtype, cudaStream_t q) {
    plan_tiles(a, GV_ROWS);
    if (dtype == DET_BF16) launch_mt<bf16>(a, q);
    else launch_mt<float>(a, q);
}

// `rows` input rows become the groups of a one-row call.
static FgemmArgs group_args(FgemmArgs a, int rows) {
    a.M = 1;
    a.nseg = 1;
    a.seg_end[0] = a.N;
    a.seg_in[0] = rows - 1;
    a.gstride = a.ldx;
    return a;
}
bool fgemv_group_takes(const FgemmArgs& a, int rows) {
    if (float_flags() & 2) return false;
    return rows <= 4 && gemv_smem(group_args(a, rows), 1) <= smem_optin() - 8192;
}
void fgemv_group_launch(FgemmArgs a, int dtype, cudaStream_t q) {
    a = group_args(a, a.pairs / a.pairs_per_row);
    if (dtype == DET_BF16) launch_gemv<bf16, 1, false, true>(a, q);
    else launch_gemv<float, 1, false, true>(a, q);
}

}  // namespace detb
