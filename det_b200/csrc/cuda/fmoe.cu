// Mixture of experts (include/det_b200.h, det_fmoe_op): softmax router with a correction that only chooses, weights of the chosen
// scaled to one, experts of the form W_down max(W_up x, 0)^2, identity experts, one shared expert behind a gate.
//
//   k_fmoe_route    a warp per row: softmax, the `top` largest choice scores, weights; counts the rows of every expert.
// Few rows (decode): every (row, expert) pair streams its expert's weights once,
//   k_fgemv         first halves, a quad of weight rows belonging to a pair;
//   k_fmoe_down     a row's chosen second halves as one product over the concatenated activations, weights, shared expert and
//                   identity experts included.  Both bound by the bytes of the chosen experts.
// More rows: pairs are sorted by expert,
//   k_fmoe_gather   prefix sums over the counts, the work list of the products, the rows in order of their expert;
//   k_fgemm_tc / k_fgemm_simt over the work list, both halves;
//   k_fmoe_combine  a row's weighted sum.  A pair's place does not enter its value and a row adds its pairs in the order they
//                   were chosen, so results do not depend on what else is in the batch.
#include "fops.cuh"
#include <algorithm>

namespace detb {

struct MoeArgs {
    int experts, outputs, top, ff, n, M;
    const float* z;
    int ldz;
    const float* correction;
    const void* x;
    int ldx;
    const bf16* down;
    int ldd;
    const bf16* sdown;          // shared second half, or NULL
    int sk, lds;
    const void* hs;
    int ldhs, shared_gate;
    float* out;
    int ldo;
    unsigned* counts;
    // scratch
    int* sel;                   // [M][top] chosen outputs
    float* weight;              // [M][top]
    int* rank;                  // [M][top] place among the expert's rows, then place among all rows (-1: identity)
    float* extra;               // [M][2] weight of x itself, gate of the shared expert
    int* nwork;
    int4* work;
    void* xp;                   // [M * top][ldx] rows in order of their expert
    void* h1;                   // [M * top][ldh] first halves
    int ldh;
    float* yp;                  // [M * top][n]
    int tok;                    // rows per work entry
};

// ------------------------------------------------------------------------------------------------------ routing
// Order-preserving integer image of a float.
__device__ __forceinline__ unsigned key_of(float v) {
    const unsigned b = __float_as_uint(v);
    return (b & 0x80000000u) ? ~b : b | 0x80000000u;
}
constexpr int ROUTE_WARPS = 4;
template <int NL>      // outputs per lane
__global__ void __launch_bounds__(ROUTE_WARPS * 32) k_fmoe_route(const MoeArgs a, int sorted) {
    pdl_trigger();
    pdl_wait();
    const int row = blockIdx.x * ROUTE_WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (row >= a.M) return;
    const float* z = a.z + (size_t)row * a.ldz;
    float s[NL];
    float m = -INFINITY;
#pragma unroll
    for (int i = 0; i < NL; i++) {
        const int e = i * 32 + lane;
        s[i] = e < a.outputs ? z[e] : -INFINITY;
        m = fmaxf(m, s[i]);
    }
    m = warp_max(m);
    float l = 0.0f;
#pragma unroll
    for (int i = 0; i < NL; i++) {
        s[i] = expf(s[i] - m);
        l += s[i];
    }
    l = warp_sum(l);
    unsigned key[NL];
#pragma unroll
    for (int i = 0; i < NL; i++) {
        const int e = i * 32 + lane;
        s[i] /= l;
        key[i] = e < a.outputs ? key_of(s[i] + (a.correction ? a.correction[e] : 0.0f)) : 0u;
    }
    float total = 0.0f, identity = 0.0f;
    int* sel = a.sel + (size_t)row * a.top;
    float* weight = a.weight + (size_t)row * a.top;
    for (int k = 0; k < a.top; k++) {
        unsigned best = 0;
#pragma unroll
        for (int i = 0; i < NL; i++) best = max(best, key[i]);
        const unsigned win = __reduce_max_sync(FULL, best);
        const int owner = __ffs(__ballot_sync(FULL, best == win)) - 1;
        float v = 0.0f;
        int e = 0;
        if (lane == owner) {
            bool found = false;
#pragma unroll
            for (int i = 0; i < NL; i++)
                if (!found && key[i] == win) {
                    found = true;
                    v = s[i];
                    e = i * 32 + lane;
                    key[i] = 0;
                }
        }
        v = __shfl_sync(FULL, v, owner);
        e = __shfl_sync(FULL, e, owner);
        total += v;
        if (e >= a.experts) identity += v;
        if (lane == 0) {
            sel[k] = e;
            weight[k] = v;
        }
    }
    const float inv = 1.0f / (total + 1e-20f);
    __syncwarp();
    for (int k = lane; k < a.top; k += 32) {
        const int e = sel[k];
        weight[k] *= inv;
        if (sorted) a.rank[(size_t)row * a.top + k] = e < a.experts ? (int)atomicAdd(a.counts + e, 1u) : -1;
    }
    if (lane == 0) {
        a.extra[row * 2] = identity * inv;
        a.extra[row * 2 + 1] = a.shared_gate >= 0 ? sigmoid_fast(z[a.shared_gate]) : 1.0f;
    }
}

// ------------------------------------------------------------------------------------------------------ few rows
constexpr int MD_WARPS = 16, MD_THREADS = MD_WARPS * 32, MD_ROWS = 4, MD_MAX = 64;   // MD_MAX: second halves of a row

__device__ __forceinline__ void load_eight(const float* p, float (&v)[8]) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
    v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void load_eight(const bf16* p, float (&v)[8]) {
    const uint4 a = *reinterpret_cast<const uint4*>(p);
    v[0] = bf_lo(a.x); v[1] = bf_hi(a.x); v[2] = bf_lo(a.y); v[3] = bf_hi(a.y);
    v[4] = bf_lo(a.z); v[5] = bf_hi(a.z); v[6] = bf_lo(a.w); v[7] = bf_hi(a.w);
}

// grid (CTAs, rows).  xs: the row's weighted first halves side by side, each padded to a multiple of 8, two planes of four.
template <class T>
__global__ void __launch_bounds__(MD_THREADS, 1) k_fmoe_down(const MoeArgs a, int wsplit) {
    extern __shared__ __align__(16) float xs[];
    __shared__ const bf16* base[MD_MAX];
    __shared__ int ld[MD_MAX], start[MD_MAX + 1], from[MD_MAX];
    __shared__ float scale[MD_MAX];
    __shared__ float red[2][MD_WARPS][MD_ROWS];
    __shared__ int count;
    pdl_trigger();
    pdl_wait();
    const int row = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int* sel = a.sel + (size_t)row * a.top;
    const float* extra = a.extra + row * 2;
    const int fp = (a.ff + 7) & ~7, sp = (a.sk + 7) & ~7;
    // the segments of the row's product: its chosen experts in order, then the shared one
    if (warp == 0) {
        int c = 0;
        for (int k0 = 0; k0 < a.top; k0 += 32) {
            const int k = k0 + lane, e = k < a.top ? sel[k] : a.experts;
            const unsigned real = __ballot_sync(FULL, e < a.experts);
            if (e < a.experts) {
                const int i = c + __popc(real & ((1u << lane) - 1u));
                base[i] = a.down + (size_t)e * a.n * a.ldd;
                ld[i] = a.ldd;
                start[i] = i * fp;
                from[i] = k;
                scale[i] = a.weight[(size_t)row * a.top + k];
            }
            c += __popc(real);
        }
        if (lane == 0) {
            start[c] = c * fp;
            if (a.sdown) {
                base[c] = a.sdown;
                ld[c] = a.lds;
                from[c] = -1;
                scale[c] = extra[1];
                c++;
                start[c] = start[c - 1] + sp;
            }
            count = c;
        }
    }
    __syncthreads();
    const int nseg = count, kt = start[nseg], half = kt / 2;
    const int group = warp / wsplit, part = warp % wsplit, qpc = MD_WARPS / wsplit;
    const int nquads = (a.n + MD_ROWS - 1) / MD_ROWS, stride = qpc * gridDim.x, kstep = wsplit * 256;
    int quad = blockIdx.x * qpc + group, buf = 0, seg = 0;
    const int k_first = (part * 32 + lane) * 8;
    auto load = [&](int qd, int k, uint4 (&w)[MD_ROWS]) {
        if (k >= kt || qd >= nquads) {
#pragma unroll
            for (int r = 0; r < MD_ROWS; r++) w[r] = make_uint4(0, 0, 0, 0);
            return;
        }
        while (k >= start[seg + 1]) seg++;
        const bf16* p = base[seg] + (k - start[seg]);
        const size_t l = ld[seg];
#pragma unroll
        for (int r = 0; r < MD_ROWS; r++) w[r] = __ldcs(reinterpret_cast<const uint4*>(p + min(qd * MD_ROWS + r, a.n - 1) * l));
    };
    uint4 w0[MD_ROWS], w1[MD_ROWS];
    load(quad, k_first, w0);
    {
        int s = 0;
        for (int j = threadIdx.x * 8; j < kt; j += MD_THREADS * 8) {
            while (j >= start[s + 1]) s++;
            const int i = j - start[s], n = (from[s] < 0 ? a.sk : a.ff) - i;
            const T* h = from[s] < 0 ? static_cast<const T*>(a.hs) + (size_t)row * a.ldhs : static_cast<const T*>(a.h1) + ((size_t)row * a.top + from[s]) * a.ldh;
            float v[8];
            load_eight(h + i, v);
#pragma unroll
            for (int t = 0; t < 8; t++) v[t] = t < n ? v[t] * scale[s] : 0.0f;
            *reinterpret_cast<float4*>(xs + (j >> 1)) = make_float4(v[0], v[1], v[2], v[3]);
            *reinterpret_cast<float4*>(xs + half + (j >> 1)) = make_float4(v[4], v[5], v[6], v[7]);
        }
    }
    const float identity = extra[0];
    __syncthreads();
    for (int b = blockIdx.x * qpc; b < nquads; b += stride, quad += stride, buf ^= 1) {
        const bool live = quad < nquads;
        if (live) {
            float acc[MD_ROWS] = {0.0f, 0.0f, 0.0f, 0.0f};
            for (int k = k_first; k < kt; k += kstep) {
                if (k + kstep < kt) {
                    load(quad, k + kstep, w1);
                } else {                              // the next quad's first weights, ahead of this one's sums
                    seg = 0;
                    load(quad + stride, k_first, w1);
                }
                const float4 xa = *reinterpret_cast<const float4*>(xs + (k >> 1)), xb = *reinterpret_cast<const float4*>(xs + half + (k >> 1));
#pragma unroll
                for (int r = 0; r < MD_ROWS; r++) {
                    float s = acc[r];
                    s = fmaf(bf_lo(w0[r].x), xa.x, s);
                    s = fmaf(bf_hi(w0[r].x), xa.y, s);
                    s = fmaf(bf_lo(w0[r].y), xa.z, s);
                    s = fmaf(bf_hi(w0[r].y), xa.w, s);
                    s = fmaf(bf_lo(w0[r].z), xb.x, s);
                    s = fmaf(bf_hi(w0[r].z), xb.y, s);
                    s = fmaf(bf_lo(w0[r].w), xb.z, s);
                    s = fmaf(bf_hi(w0[r].w), xb.w, s);
                    acc[r] = s;
                    w0[r] = w1[r];
                }
            }
#pragma unroll
            for (int r = 0; r < MD_ROWS; r++) {
                const float s = warp_sum(acc[r]);
                if (lane == 0) red[buf][warp][r] = s;
            }
        }
        if (wsplit == 1) __syncwarp();
        else if (wsplit == MD_WARPS) __syncthreads();
        else asm volatile("bar.sync %0, %1;" ::"r"(1 + group), "r"(wsplit * 32) : "memory");
        if (live && part == 0 && lane < MD_ROWS) {
            const int n = quad * MD_ROWS + lane;
            if (n < a.n) {
                float v = 0.0f;
                for (int i = 0; i < wsplit; i++) v += red[buf][group * wsplit + i][lane];
                if (identity != 0.0f) v = fmaf(identity, to_f(static_cast<const T*>(a.x)[(size_t)row * a.ldx + n]), v);
                a.out[(size_t)row * a.ldo + n] = v;
            }
        }
    }
}

// ------------------------------------------------------------------------------------------------------ more rows
constexpr int MG_WARPS = 8;
// First row of every expert among the sorted rows, and its first work entry.
__device__ __forceinline__ void expert_offsets(const MoeArgs& a, int* off, int* entry) {
    if (threadIdx.x < 32) {
        const int lane = threadIdx.x;
        int rows = 0, entries = 0;
        for (int e0 = 0; e0 < a.experts; e0 += 32) {
            const int c = e0 + lane < a.experts ? (int)a.counts[e0 + lane] : 0, t = (c + a.tok - 1) / a.tok;
            int rs = c, es = t;
#pragma unroll
            for (int d = 1; d < 32; d <<= 1) {
                const int r = __shfl_up_sync(FULL, rs, d), w = __shfl_up_sync(FULL, es, d);
                if (lane >= d) {
                    rs += r;
                    es += w;
                }
            }
            if (e0 + lane < a.experts) {
                off[e0 + lane] = rows + rs - c;
                entry[e0 + lane] = entries + es - t;
            }
            rows += __shfl_sync(FULL, rs, 31);
            entries += __shfl_sync(FULL, es, 31);
        }
        if (lane == 0) {
            off[a.experts] = rows;
            entry[a.experts] = entries;
        }
    }
    __syncthreads();
}
template <class T>
__global__ void __launch_bounds__(MG_WARPS * 32) k_fmoe_gather(const MoeArgs a) {
    __shared__ int off[DET_MAX_ROUTER + 1], entry[DET_MAX_ROUTER + 1];
    pdl_trigger();
    pdl_wait();
    expert_offsets(a, off, entry);
    if (blockIdx.x == 0) {
        for (int e = threadIdx.x; e < a.experts; e += MG_WARPS * 32)
            for (int i = entry[e], r = off[e]; i < entry[e + 1]; i++, r += a.tok) a.work[i] = make_int4(e, r, min(r + a.tok, off[e + 1]), 0);
        if (threadIdx.x == 0) *a.nwork = entry[a.experts];
    }
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, pair = blockIdx.x * MG_WARPS + warp;
    if (pair >= a.M * a.top) return;
    const int e = a.sel[pair];
    if (e >= a.experts) return;
    const int place = off[e] + a.rank[pair];
    __syncwarp();
    if (lane == 0) a.rank[pair] = place;
    constexpr int VEC = 16 / sizeof(T);
    const uint4* src = reinterpret_cast<const uint4*>(static_cast<const T*>(a.x) + (size_t)(pair / a.top) * a.ldx);
    uint4* dst = reinterpret_cast<uint4*>(static_cast<T*>(a.xp) + (size_t)place * a.ldx);
    for (int i = lane; i < a.ldx / VEC; i += 32) dst[i] = src[i];
    // the products read whole 16-byte pieces of the first halves
    T* h = static_cast<T*>(a.h1) + (size_t)place * a.ldh;
    for (int i = a.ff + lane; i < a.ldh; i += 32) put(h + i, 0.0f);
}

// out holds the shared expert's second half when there is one.  V columns per thread and pass.
template <class T, int V>
__global__ void __launch_bounds__(256) k_fmoe_combine(const MoeArgs a) {
    __shared__ int rows[DET_MAX_ROUTER];
    __shared__ float weights[DET_MAX_ROUTER];
    pdl_trigger();
    pdl_wait();
    const int row = blockIdx.x;
    if (row == 0 && blockIdx.y == 0)
        for (int e = threadIdx.x; e < a.experts; e += 256) a.counts[e] = 0;     // for the next call
    for (int k = threadIdx.x; k < a.top; k += 256) {
        const int p = a.rank[(size_t)row * a.top + k];
        rows[k] = max(p, 0);
        weights[k] = p >= 0 ? a.weight[(size_t)row * a.top + k] : 0.0f;
    }
    const float identity = a.extra[row * 2], gate = a.extra[row * 2 + 1];
    const T* x = static_cast<const T*>(a.x) + (size_t)row * a.ldx;
    float* out = a.out + (size_t)row * a.ldo;
    __syncthreads();
    for (int i = (blockIdx.y * 256 + threadIdx.x) * V; i < a.n; i += gridDim.y * 256 * V) {
        float v[V];
#pragma unroll
        for (int j = 0; j < V; j++) v[j] = a.sdown ? gate * out[i + j] : 0.0f;
        if (identity != 0.0f)
#pragma unroll
            for (int j = 0; j < V; j++) v[j] = fmaf(identity, to_f(x[i + j]), v[j]);
#pragma unroll 4
        for (int k = 0; k < a.top; k++) {
            if (weights[k] == 0.0f) continue;                                  // x itself: no row of its own
            const float* y = a.yp + (size_t)rows[k] * a.n + i;
            if constexpr (V == 4) {
                const float4 f = *reinterpret_cast<const float4*>(y);
                v[0] = fmaf(weights[k], f.x, v[0]);
                v[1] = fmaf(weights[k], f.y, v[1]);
                v[2] = fmaf(weights[k], f.z, v[2]);
                v[3] = fmaf(weights[k], f.w, v[3]);
            } else {
                v[0] = fmaf(weights[k], *y, v[0]);
            }
        }
        if constexpr (V == 4) *reinterpret_cast<float4*>(out + i) = make_float4(v[0], v[1], v[2], v[3]);
        else out[i] = v[0];
    }
}

template <class T>
static void launch_combine(const MoeArgs& a, cudaStream_t q) {
    const bool wide = a.n % 4 == 0 && a.ldo % 4 == 0 && (reinterpret_cast<uintptr_t>(a.out) & 15) == 0;
    const int cols = 256 * (wide ? 4 : 1);
    const dim3 grid(a.M, std::max(1, std::min((a.n + cols - 1) / cols, 8 * sm_count() / a.M)));
    if (wide) launch_pdl(k_fmoe_combine<T, 4>, grid, dim3(256), 0, q, 1, a);
    else launch_pdl(k_fmoe_combine<T, 1>, grid, dim3(256), 0, q, 1, a);
}

// ------------------------------------------------------------------------------------------------------ host side
static size_t align256(size_t n) { return (n + 255) & ~(size_t)255; }
static int max_entries(int pairs, int experts, int tok) { return std::min(pairs, experts + pairs / tok); }
static size_t layout(MoeArgs& a, uint8_t* base, int esz) {
    size_t at = 0;
    auto take = [&](size_t bytes) {
        uint8_t* p = base + at;
        at += align256(bytes);
        return p;
    };
    const size_t pairs = (size_t)a.M * a.top;
    a.sel = reinterpret_cast<int*>(take(pairs * 4));
    a.weight = reinterpret_cast<float*>(take(pairs * 4));
    a.rank = reinterpret_cast<int*>(take(pairs * 4));
    a.extra = reinterpret_cast<float*>(take((size_t)a.M * 8));
    a.nwork = reinterpret_cast<int*>(take(4));
    a.work = reinterpret_cast<int4*>(take((size_t)max_entries((int)pairs, a.experts, 32) * 16));
    a.ldh = round8(a.ff);
    a.h1 = take(pairs * a.ldh * esz);
    a.xp = take(pairs * round8(a.n) * esz);
    a.yp = reinterpret_cast<float*>(take(pairs * a.n * 4));
    return at;
}
static size_t down_smem(const MoeArgs& a) { return ((size_t)a.top * round8(a.ff) + round8(a.sk)) * sizeof(float); }

template <class T>
static void launch_down(const MoeArgs& a, cudaStream_t q) {
    const size_t smem = down_smem(a);
    static size_t configured = 40 * 1024;
    if (smem > configured) {
        DETB_CUDA_OK(cudaFuncSetAttribute(k_fmoe_down<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        configured = smem;
    }
    const int quads = (a.n + MD_ROWS - 1) / MD_ROWS, sms = std::max(1, sm_count() / a.M), kt = a.top * round8(a.ff) + round8(a.sk);
    int wsplit = 1;
    double best = 1e30;
    for (int ws = 1; ws <= MD_WARPS; ws *= 2) {
        if (ws > 1 && (ws - 1) * 256 >= kt) break;
        const int per_round = sms * (MD_WARPS / ws);
        const double cost = (double)((quads + per_round - 1) / per_round) * (1.0 / ws) * (1.0 + 0.02 * ws);
        if (cost < best * 0.999) {
            best = cost;
            wsplit = ws;
        }
    }
    const int qpc = MD_WARPS / wsplit;
    launch_pdl(k_fmoe_down<T>, dim3(std::min(sms, (quads + qpc - 1) / qpc), a.M), dim3(MD_THREADS), smem, q, 1, a, wsplit);
}

}  // namespace detb

using namespace detb;

extern "C" {

size_t det_f_moe_scratch_bytes(int M, int experts, int top, int ff, int n, int dtype) {
    MoeArgs a{};
    a.M = M; a.experts = experts; a.top = top; a.ff = ff; a.n = n;
    return layout(a, nullptr, dtype == DET_BF16 ? 2 : 4) + 256;
}

void det_f_moe(const det_fmoe_op* op, cudaStream_t st) {
    const int outputs = op->experts + op->identity;
    DETB_REQUIRE(op->experts > 0 && op->identity >= 0 && outputs <= DET_MAX_ROUTER && op->top > 0 && op->top <= outputs && op->ff > 0 && op->n > 0,
                 "mixture: bad sizes");
    DETB_REQUIRE(op->up->N == op->experts * op->ff && op->up->K == op->n && op->down->N == op->experts * op->n && op->down->K == op->ff,
                 "mixture: the experts' weights do not fit");
    DETB_REQUIRE(op->ldx == round8(op->n) || op->M <= 0, "mixture: bad input rows");
    DETB_REQUIRE(!op->shared || (op->hs && op->shared->N == op->n && op->ldhs >= op->shared->ld), "mixture: bad shared expert");
    if (op->M <= 0) return;
    MoeArgs a{};
    a.experts = op->experts; a.outputs = outputs; a.top = op->top; a.ff = op->ff; a.n = op->n; a.M = op->M;
    a.z = op->z; a.ldz = op->ldz; a.correction = op->correction;
    a.x = op->x; a.ldx = op->ldx;
    a.down = static_cast<const bf16*>(op->down->w);
    a.ldd = op->down->ld;
    if (op->shared) {
        a.sdown = static_cast<const bf16*>(op->shared->w);
        a.sk = op->shared->K;
        a.lds = op->shared->ld;
    }
    a.hs = op->hs; a.ldhs = op->ldhs; a.shared_gate = op->shared_gate;
    a.out = op->out; a.ldo = op->ldo; a.counts = op->counts;
    const bool bf = op->dtype == DET_BF16;
    layout(a, static_cast<uint8_t*>(op->scratch), bf ? 2 : 4);
    cudaStream_t q = queue_of(st);
    const int pairs = a.M * a.top;

    FgemmArgs up{};
    up.w = static_cast<const bf16*>(op->up->w);
    up.wt = static_cast<const bf16*>(op->up->wt);
    up.N = op->up->N; up.K = op->up->K; up.ldw = op->up->ld;
    up.x = op->x; up.ldx = op->ldx;
    up.nseg = 1;
    up.seg_end[0] = up.N;
    up.act = DET_FF_RELU2;
    up.h = a.h1; up.ldh = a.ldh;
    up.group_rows = op->ff;
    up.groups = op->experts;
    up.error_flag = error_word();
    up.sel = a.sel;
    up.pairs = pairs;
    up.pairs_per_row = a.top;
    const bool few = a.M <= 4 && a.top < MD_MAX && down_smem(a) <= smem_optin() - 8192 && fgemv_group_takes(up, a.M);

    const dim3 rgrid((a.M + ROUTE_WARPS - 1) / ROUTE_WARPS), rblock(ROUTE_WARPS * 32);
    if (outputs <= 64) launch_pdl(k_fmoe_route<2>, rgrid, rblock, 0, q, 1, a, few ? 0 : 1);
    else if (outputs <= 128) launch_pdl(k_fmoe_route<4>, rgrid, rblock, 0, q, 1, a, few ? 0 : 1);
    else if (outputs <= 256) launch_pdl(k_fmoe_route<8>, rgrid, rblock, 0, q, 1, a, few ? 0 : 1);
    else launch_pdl(k_fmoe_route<32>, rgrid, rblock, 0, q, 1, a, few ? 0 : 1);
    if (few) {
        fgemv_group_launch(up, op->dtype, q);
        if (bf) launch_down<bf16>(a, q);
        else launch_down<float>(a, q);
        return;
    }
    DETB_REQUIRE(op->counts, "mixture: no counters");
    a.tok = fgemm_group_tok(op->dtype, pairs / op->experts);
    const dim3 ggrid((pairs + MG_WARPS - 1) / MG_WARPS), gblock(MG_WARPS * 32);
    if (bf) launch_pdl(k_fmoe_gather<bf16>, ggrid, gblock, 0, q, 1, a);
    else launch_pdl(k_fmoe_gather<float>, ggrid, gblock, 0, q, 1, a);
    up.x = a.xp;
    up.M = pairs;
    up.work = a.work;
    up.nwork = a.nwork;
    up.max_work = max_entries(pairs, op->experts, a.tok);
    fgemm_group_launch(up, op->dtype, a.tok, q);
    FgemmArgs dn = up;
    dn.w = a.down;
    dn.wt = static_cast<const bf16*>(op->down->wt);
    dn.N = op->down->N; dn.K = op->down->K; dn.ldw = op->down->ld;
    dn.x = a.h1; dn.ldx = a.ldh;
    dn.seg_end[0] = dn.N;
    dn.glu_from = dn.N;
    dn.act = 0;
    dn.h = nullptr;
    dn.y = a.yp; dn.ldy = a.n;
    dn.group_rows = op->n;
    fgemm_group_launch(dn, op->dtype, a.tok, q);
    if (op->shared) {
        det_fgemm_op g{};
        g.lin = op->shared;
        g.dtype = op->dtype;
        g.x = op->hs;
        g.ldx = op->ldhs;
        g.nseg = 1;
        g.seg_end[0] = op->n;
        g.glu_from = op->n;
        g.M = op->M;
        g.y = op->out;
        g.ldy = op->ldo;
        det_f_gemm(&g, st);
    }
    if (bf) launch_combine<bf16>(a, q);
    else launch_combine<float>(a, q);
}

}  // extern "C"
