// The seam between two sublayers (include/det_b200.h, det_fseam_op): norm of the sublayer's result, layer scale, residual add,
// norm of the new row and a short causal convolution over time, all on fp32 residual rows.
//
//   k_fseam   a row per cluster of up to eight CTAs (one for long runs of rows): the two sums of squares cross the cluster through
//             distributed shared memory, so that a decoded token's seam is one launch and not one CTA's work.  The convolution
//             runs here when every row has a history of its own (decode, batches).
//   k_fconv   the convolution over a run of tokens: reciprocal norms come from k_fseam, a thread walks 16 rows of its
//             columns with the earlier rows in registers.  Both forms convolve fp32 values, so a cut of the run does not show.
#include "fops.cuh"
#include <algorithm>
#include <cooperative_groups.h>

namespace detb {

constexpr int SEAM_THREADS = 256, SEAM_MAX_CLUSTER = 8;

template <int V>
struct Vec {
    float v[V];
};
template <int V>
__device__ __forceinline__ Vec<V> load_vec(const float* p) {
    Vec<V> r;
    if constexpr (V == 4) {
        const float4 f = *reinterpret_cast<const float4*>(p);
        r.v[0] = f.x; r.v[1] = f.y; r.v[2] = f.z; r.v[3] = f.w;
    } else {
        r.v[0] = *p;
    }
    return r;
}
template <int V>
__device__ __forceinline__ void store_vec(float* p, const Vec<V>& r) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else *p = r.v[0];
}
template <int V>
__device__ __forceinline__ void store_vec(bf16* p, const Vec<V>& r) {
    if constexpr (V == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf(r.v[0], r.v[1]), pack_bf(r.v[2], r.v[3]));
    else put(p, r.v[0]);
}

// Sum over the row's cluster.  Every CTA pushes its part to all peers, so none reads a peer that may have left.
__device__ __forceinline__ float row_sum(float v, float* sh, float* slots, int cs) {
    namespace cg = cooperative_groups;
    v = block_sum(v, sh);
    if (cs == 1) return v;
    cg::cluster_group cl = cg::this_cluster();
    if ((int)threadIdx.x < cs) *cl.map_shared_rank(slots + cl.block_rank(), threadIdx.x) = v;
    cl.sync();
    float s = 0.0f;
    for (int i = 0; i < cs; i++) s += slots[i];
    return s;
}

// `own`: every row of the call has its own history (or the call is one row).  ONE: a thread has one vector of the row, which
// stays in registers, and loads what does not depend on the kernel before ahead of the wait; otherwise the row goes through
// shared memory, which leaves room for eight CTAs an SM.
template <class T, int V, bool ONE>
__global__ void __launch_bounds__(SEAM_THREADS) k_fseam(const det_fseam_op a, int cs, int own) {
    extern __shared__ __align__(16) float buf[];        // this CTA's columns
    __shared__ float sh[32];
    __shared__ float slots[2][SEAM_MAX_CLUSTER];
    pdl_trigger();
    const int row = blockIdx.x / cs, piece = blockIdx.x % cs;
    const int per = ((a.n + V - 1) / V + cs - 1) / cs * V, c0 = min(a.n, piece * per), c1 = min(a.n, c0 + per);
    const int first = c0 + (int)threadIdx.x * V;
    float* x = a.x + (size_t)row * a.n;
    auto each = [&](auto f) {
        if constexpr (ONE) {
            if (first < c1) f(first);
        } else {
            for (int i = first; i < c1; i += SEAM_THREADS * V) f(i);
        }
    };
    Vec<V> mine, xv, yn, ys, w;
    auto keep = [&](int i, const Vec<V>& v) {
        if constexpr (ONE) mine = v;
        else store_vec(buf + (i - c0), v);
    };
    auto kept = [&](int i) {
        if constexpr (ONE) return mine;
        else return load_vec<V>(buf + (i - c0));
    };
    if constexpr (ONE)
        each([&](int i) {
            if (a.y) yn = load_vec<V>(a.y_norm + i);
            if (a.y && a.y_scale) ys = load_vec<V>(a.y_scale + i);
            if (a.w) w = load_vec<V>(a.w + i);
        });
    if (cs > 1) cooperative_groups::this_cluster().sync();      // peers run before anything is pushed to them
    pdl_wait();
    if constexpr (ONE) each([&](int i) { xv = load_vec<V>(x + i); });
    float ss = 0.0f;
    if (a.y) {
        const float* y = a.y + (size_t)row * a.ldy;
        each([&](int i) {
            const Vec<V> v = load_vec<V>(y + i);
#pragma unroll
            for (int j = 0; j < V; j++) ss = fmaf(v.v[j], v.v[j], ss);
            keep(i, v);
        });
        const float rs = 1.0f / sqrtf(row_sum(ss, sh, slots[0], cs) / (float)a.n + a.eps);
        ss = 0.0f;
        each([&](int i) {
            const Vec<V> v = kept(i);
            if constexpr (!ONE) {
                xv = load_vec<V>(x + i);
                yn = load_vec<V>(a.y_norm + i);
                if (a.y_scale) ys = load_vec<V>(a.y_scale + i);
            }
            Vec<V> r = xv;
#pragma unroll
            for (int j = 0; j < V; j++) {
                float t = v.v[j] * rs * yn.v[j];
                if (a.y_scale) t *= ys.v[j];
                r.v[j] += t;
                ss = fmaf(r.v[j], r.v[j], ss);
            }
            store_vec(x + i, r);
            keep(i, r);
        });
    } else {
        each([&](int i) {
            const Vec<V> v = ONE ? xv : load_vec<V>(x + i);
#pragma unroll
            for (int j = 0; j < V; j++) ss = fmaf(v.v[j], v.v[j], ss);
            keep(i, v);
        });
    }
    if (!a.out) return;
    float rs = 1.0f;
    if (a.w) rs = 1.0f / sqrtf(row_sum(ss, sh, slots[1], cs) / (float)a.n + a.eps);
    if (a.conv && !own) {
        if (piece == 0 && threadIdx.x == 0) a.rstd[row] = rs;
        return;
    }
    T* out = static_cast<T*>(a.out) + (size_t)row * a.ld;
    float* prev = a.conv ? slot_of(a.seq, row).prev : nullptr;
    each([&](int i) {
        Vec<V> h = kept(i);
        if (a.w) {
            if constexpr (!ONE) w = load_vec<V>(a.w + i);
#pragma unroll
            for (int j = 0; j < V; j++) h.v[j] = h.v[j] * rs * w.v[j];
        }
        if (a.conv) {
            Vec<V> o = h;
#pragma unroll 4
            for (int t = 0; t < a.taps - 1; t++) {
                const Vec<V> p = load_vec<V>(prev + (size_t)t * a.n + i), c = load_vec<V>(a.conv + (size_t)t * a.n + i);
#pragma unroll
                for (int j = 0; j < V; j++) o.v[j] = fmaf(c.v[j], p.v[j], o.v[j]);
                if (t > 0) store_vec(prev + (size_t)(t - 1) * a.n + i, p);
            }
            const Vec<V> c = load_vec<V>(a.conv + (size_t)(a.taps - 1) * a.n + i);
            if (a.taps > 1) store_vec(prev + (size_t)(a.taps - 2) * a.n + i, h);
#pragma unroll
            for (int j = 0; j < V; j++) o.v[j] = fmaf(c.v[j], h.v[j], o.v[j]);
            h = o;
        }
        store_vec(out + i, h);
    });
}

// ---------------------------------------------------------------------------------------------- runs of tokens
constexpr int CONV_ROWS = DET_MAX_TAPS;      // rows of a thread: at least the history's, so that only the first run reads prev

// TP: taps rounded up; missing leading taps weigh zero.
template <class T, int V, int TP>
__global__ void __launch_bounds__(SEAM_THREADS) k_fconv(const det_fseam_op a) {
    pdl_trigger();
    pdl_wait();
    const int i = (blockIdx.y * SEAM_THREADS + threadIdx.x) * V;
    if (i >= a.n) return;
    const int r0 = blockIdx.x * CONV_ROWS, r1 = min(a.M, r0 + CONV_ROWS), lead = TP - a.taps;
    const Vec<V> w = load_vec<V>(a.w + i);
    auto normed = [&](int r) {
        Vec<V> h = load_vec<V>(a.x + (size_t)r * a.n + i);
        const float rs = a.rstd[r];
#pragma unroll
        for (int j = 0; j < V; j++) h.v[j] = h.v[j] * rs * w.v[j];
        return h;
    };
    Vec<V> c[TP], past[TP - 1];
#pragma unroll
    for (int t = 0; t < TP; t++) {
        if (t >= lead) c[t] = load_vec<V>(a.conv + (size_t)(t - lead) * a.n + i);
        else
#pragma unroll
            for (int j = 0; j < V; j++) c[t].v[j] = 0.0f;
    }
    float* prev = a.seq.one.prev;
#pragma unroll
    for (int t = 0; t < TP - 1; t++) {
        if (t < lead) past[t] = c[0];                       // zeros when lead > 0
        else if (r0 > 0) past[t] = normed(r0 - (TP - 1) + t);
        else past[t] = load_vec<V>(prev + (size_t)(t - lead) * a.n + i);
    }
    for (int r = r0; r < r1; r++) {
        const Vec<V> h = normed(r);
        Vec<V> o = h;
#pragma unroll
        for (int t = 0; t < TP - 1; t++)
#pragma unroll
            for (int j = 0; j < V; j++) o.v[j] = fmaf(c[t].v[j], past[t].v[j], o.v[j]);
#pragma unroll
        for (int j = 0; j < V; j++) o.v[j] = fmaf(c[TP - 1].v[j], h.v[j], o.v[j]);
#pragma unroll
        for (int t = 0; t + 1 < TP - 1; t++) past[t] = past[t + 1];
        past[TP - 2] = h;
        store_vec(static_cast<T*>(a.out) + (size_t)r * a.ld + i, o);
    }
    if (r0 > 0) return;
    // the thread that has read the old history writes the new one
#pragma unroll
    for (int t = 0; t < TP - 1; t++) {
        if (t < lead) continue;
        const Vec<V> h = a.M > CONV_ROWS ? normed(a.M - (TP - 1) + t) : past[t];
        store_vec(prev + (size_t)(t - lead) * a.n + i, h);
    }
}

template <class T, int V, bool ONE>
static void launch_row(const det_fseam_op& op, int cs, int own, cudaStream_t q) {
    size_t smem = 0;
    if constexpr (!ONE) {
        smem = (size_t)(((op.n + V - 1) / V + cs - 1) / cs * V) * sizeof(float);
        static size_t configured = 48 * 1024;
        if (smem > configured) {
            DETB_CUDA_OK(cudaFuncSetAttribute(k_fseam<T, V, ONE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
            configured = smem;
        }
    }
    launch_pdl(k_fseam<T, V, ONE>, dim3(op.M * cs), dim3(SEAM_THREADS), smem, q, cs, op, cs, own);
}
template <class T, int V>
static void launch_seam(const det_fseam_op& op, cudaStream_t q) {
    const bool own = op.seq.table != nullptr || op.M == 1 || !op.conv;
    auto vecs = [&](int cs) { return ((op.n + V - 1) / V + cs - 1) / cs; };      // of a CTA
    int cs = 1;
    while (cs < SEAM_MAX_CLUSTER && vecs(cs) > SEAM_THREADS && (long long)op.M * cs * 2 <= sm_count()) cs *= 2;
    if (vecs(cs) <= SEAM_THREADS) launch_row<T, V, true>(op, cs, own ? 1 : 0, q);
    else launch_row<T, V, false>(op, cs, own ? 1 : 0, q);
    if (own || !op.out) return;
    if (op.taps <= 4) {
        launch_pdl(k_fconv<T, V, 4>, dim3((op.M + CONV_ROWS - 1) / CONV_ROWS, (op.n + SEAM_THREADS * V - 1) / (SEAM_THREADS * V)),
                   dim3(SEAM_THREADS), 0, q, 1, op);
    } else {
        launch_pdl(k_fconv<T, 1, DET_MAX_TAPS>, dim3((op.M + CONV_ROWS - 1) / CONV_ROWS, (op.n + SEAM_THREADS - 1) / SEAM_THREADS),
                   dim3(SEAM_THREADS), 0, q, 1, op);
    }
}

}  // namespace detb

using namespace detb;

extern "C" void det_f_seam(const det_fseam_op* op, cudaStream_t st) {
    DETB_REQUIRE(op->x && op->n > 0 && (!op->y || (op->y_norm && op->ldy >= op->n)), "seam: bad input");
    DETB_REQUIRE(!op->out || (op->ld % 8 == 0 && op->ld >= op->n), "seam: bad output rows");
    DETB_REQUIRE(!op->conv || (op->w && op->taps >= 1 && op->taps <= DET_MAX_TAPS), "seam: bad convolution");
    if (op->M <= 0) return;
    DETB_REQUIRE(!op->conv || op->seq.table || op->M == 1 || op->rstd, "seam: a run of tokens needs scratch");
    DETB_REQUIRE((size_t)op->n * sizeof(float) <= smem_optin() - 4096, "seam: the row is too long");
    auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    // four columns at a time where every row allows it
    const bool wide = op->n % 4 == 0 && op->ldy % 4 == 0 && aligned(op->x) && aligned(op->y) && aligned(op->y_norm) && aligned(op->y_scale) &&
                      aligned(op->w) && aligned(op->conv) && aligned(op->out) && (op->seq.table || aligned(op->seq.one.prev));
    cudaStream_t q = queue_of(st);
    if (op->dtype == DET_BF16) {
        if (wide) launch_seam<bf16, 4>(*op, q);
        else launch_seam<bf16, 1>(*op, q);
    } else {
        if (wide) launch_seam<float, 4>(*op, q);
        else launch_seam<float, 1>(*op, q);
    }
}
