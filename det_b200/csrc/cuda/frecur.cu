// Linear recurrences with a decay per key channel (gated linear attention and RWKV-style time mixing share one recurrence:
// include/det_b200.h, det_frecur_op).  State S[dk][dv] per head in fp32, updated in fp32.
//
//   k_frecur_step   one token per row (decode; rows may belong to different sequences): one CTA per (head, row) computes the
//                   decay from its low-rank projection, streams the head's state once, and finishes with the head's RMS norm
//                   and gate, so a layer step is one launch.  Bound by the bytes of the states.
//   k_frecur_scan   a run of tokens of one sequence: a lane keeps RPL rows of CPL columns of S in registers, PARTS lanes share
//                   a column; per-token operands are staged in shared memory in double-buffered blocks.  Bound by the latency
//                   of the token loop.  The decays come from k_fdecay, the norm and the gate from k_frecur_out.
#include "fops.cuh"
#include <algorithm>

namespace detb {

struct RecurArgs {
    int heads, dk, dv, rank, M;
    const float* y;
    int ldy, q_off, k_off, v_off, gate_off, low_off;
    float q_scale;
    int decay;
    float inv_tau;
    const bf16* w2;
    int ldw2;
    const float* bias;
    const float* u;
    const float* norm;
    float eps;
    void* out;
    int ldo;
    float* z;       // scan: decays [M][heads * dk]
    float* o;       // scan: raw outputs [M][heads * dv]
    det_seq_ref seq;
};

// ------------------------------------------------------------------------------------------------------ one token per row
constexpr int RS_THREADS = 512;

template <class T>
__global__ void __launch_bounds__(RS_THREADS) k_frecur_step(const RecurArgs a) {
    extern __shared__ __align__(16) float rsm[];
    __shared__ float sh[32];
    const int h = blockIdx.x, row = blockIdx.y, dk = a.dk, dv = a.dv, tid = threadIdx.x;
    float* sq = rsm;                 // [dk]
    float* sk = sq + dk;             // [dk]
    float* sd = sk + dk;             // [dk] decay
    float* sv = sd + dk;             // [dv]
    float* st = sv + dv;             // [rank rounded up to 8]
    float* so = st + ((a.rank + 7) & ~7);   // [groups][dv]
    pdl_trigger();
    pdl_wait();
    const float* y = a.y + (size_t)row * a.ldy;
    for (int i = tid; i < ((a.rank + 7) & ~7); i += RS_THREADS) {
        const float v = i < a.rank ? y[a.low_off + i] : 0.0f;
        st[i] = a.decay == DET_DECAY_EXP ? tanhf(v) : v;
    }
    float bonus = 0.0f;
    for (int i = tid; i < dk; i += RS_THREADS) {
        const float q = y[a.q_off + h * dk + i] * a.q_scale, k = y[a.k_off + h * dk + i];
        sq[i] = q;
        sk[i] = k;
        if (a.u) bonus = fmaf(q * a.u[h * dk + i], k, bonus);
    }
    for (int j = tid; j < dv; j += RS_THREADS) sv[j] = y[a.v_off + h * dv + j];
    if (a.u) bonus = block_sum(bonus, sh);
    __syncthreads();
    // decays: four lanes per key channel
    for (int i4 = tid; i4 < dk * 4; i4 += RS_THREADS) {
        const int i = i4 >> 2, part = i4 & 3;
        const bf16* w = a.w2 + (size_t)(h * dk + i) * a.ldw2;
        float z = 0.0f;
        for (int c = part * 8; c < a.rank; c += 32) {
            const uint4 b = *reinterpret_cast<const uint4*>(w + c);
            z = fmaf(bf_lo(b.x), st[c], z);
            z = fmaf(bf_hi(b.x), st[c + 1], z);
            z = fmaf(bf_lo(b.y), st[c + 2], z);
            z = fmaf(bf_hi(b.y), st[c + 3], z);
            z = fmaf(bf_lo(b.z), st[c + 4], z);
            z = fmaf(bf_hi(b.z), st[c + 5], z);
            z = fmaf(bf_lo(b.w), st[c + 6], z);
            z = fmaf(bf_hi(b.w), st[c + 7], z);
        }
        const unsigned quad = 0xfu << (tid & 28);
        z += __shfl_xor_sync(quad, z, 1);
        z += __shfl_xor_sync(quad, z, 2);
        if (part == 0) sd[i] = decay_of(z + a.bias[h * dk + i], a.decay, a.inv_tau);
    }
    __syncthreads();
    // state: thread = column (dv rounded up to a warp) x group of rows
    float* S = slot_of(a.seq, row).s + (size_t)h * dk * dv;
    const int vp = min((dv + 31) & ~31, RS_THREADS), ng = RS_THREADS / vp, g = tid / vp;
    if (g < ng) {
        for (int j = tid % vp; j < dv; j += vp) {
            const float v = sv[j];
            float o = 0.0f;
            constexpr int U = 8;
            for (int i0 = g; i0 < dk; i0 += ng * U) {
                float s[U];
#pragma unroll
                for (int x = 0; x < U; x++) s[x] = i0 + x * ng < dk ? S[(size_t)(i0 + x * ng) * dv + j] : 0.0f;
#pragma unroll
                for (int x = 0; x < U; x++) {
                    const int i = i0 + x * ng;
                    if (i >= dk) break;
                    const float n = fmaf(sk[i], v, sd[i] * s[x]);
                    o = fmaf(sq[i], a.u ? s[x] : n, o);
                    S[(size_t)i * dv + j] = n;
                }
            }
            so[g * dv + j] = o;
        }
    }
    __syncthreads();
    float ss = 0.0f;
    for (int j = tid; j < dv; j += RS_THREADS) {
        float o = a.u ? bonus * sv[j] : 0.0f;
        for (int x = 0; x < ng; x++) o += so[x * dv + j];
        so[j] = o;
        ss = fmaf(o, o, ss);
    }
    const float rs = 1.0f / sqrtf(block_sum(ss, sh) / (float)dv + a.eps);
    T* out = static_cast<T*>(a.out) + (size_t)row * a.ldo + h * dv;
    for (int j = tid; j < dv; j += RS_THREADS)
        put(out + j, so[j] * rs * a.norm[h * dv + j] * silu_fast(y[a.gate_off + h * dv + j]));
}

// ------------------------------------------------------------------------------------------------------ a run of tokens
constexpr int SC_WARPS = 4, SC_THREADS = SC_WARPS * 32, SC_TB = 16;   // tokens per staged block

// Row r of a head, r = (i4 * PARTS + part) * 4 + j: PARTS consecutive lanes read PARTS consecutive 16-byte pieces of a staged
// vector; the dk rows are padded with zeros to PARTS * RPL.
template <int PARTS, int RPL, int CPL, bool BONUS>
__global__ void __launch_bounds__(SC_THREADS) k_frecur_scan(const RecurArgs a) {
    constexpr int ROWS = PARTS * RPL, LC = 32 / PARTS, COLS = SC_WARPS * LC * CPL;
    extern __shared__ __align__(16) float scm[];
    constexpr int TOK_FLOATS = 3 * ROWS + COLS + 4;         // q | k | decay | v | bonus
    const int h = blockIdx.y, c0 = blockIdx.x * COLS, dk = a.dk, dv = a.dv;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, part = lane % PARTS;
    const int col = (warp * LC + lane / PARTS) * CPL;        // first column of this lane inside the CTA
    pdl_trigger();
    pdl_wait();
    float* S = a.seq.one.s + (size_t)h * dk * dv;
    float s[RPL][CPL];
#pragma unroll
    for (int i = 0; i < RPL; i++)
#pragma unroll
        for (int c = 0; c < CPL; c++) {
            const int r = ((i / 4) * PARTS + part) * 4 + (i & 3), j = c0 + col + c;
            s[i][c] = (r < dk && j < dv) ? S[(size_t)r * dv + j] : 0.0f;
        }
    // one warp stages one token at a time
    auto stage = [&](int t0, float* buf) {
        for (int t = warp; t < SC_TB && t0 + t < a.M; t += SC_WARPS) {
            const float* y = a.y + (size_t)(t0 + t) * a.ldy;
            const float* z = a.z + (size_t)(t0 + t) * a.heads * dk + h * dk;
            float* d = buf + t * TOK_FLOATS;
            float b = 0.0f;
            for (int i = lane; i < ROWS; i += 32) {
                const bool in = i < dk;
                const float q = in ? y[a.q_off + h * dk + i] * a.q_scale : 0.0f, k = in ? y[a.k_off + h * dk + i] : 0.0f;
                d[i] = q;
                d[ROWS + i] = k;
                d[2 * ROWS + i] = in ? z[i] : 0.0f;
                if (BONUS && in) b = fmaf(q * a.u[h * dk + i], k, b);
            }
            for (int j = lane; j < COLS; j += 32) d[3 * ROWS + j] = c0 + j < dv ? y[a.v_off + h * dv + c0 + j] : 0.0f;
            if (BONUS) {
                b = warp_sum(b);
                if (lane == 0) d[3 * ROWS + COLS] = b;
            }
        }
    };
    float* bufs[2] = {scm, scm + SC_TB * TOK_FLOATS};
    stage(0, bufs[0]);
    __syncthreads();
    for (int t0 = 0, p = 0; t0 < a.M; t0 += SC_TB, p ^= 1) {
        if (t0 + SC_TB < a.M) stage(t0 + SC_TB, bufs[p ^ 1]);
        const int nt = min(SC_TB, a.M - t0);
        for (int t = 0; t < nt; t++) {
            const float* d = bufs[p] + t * TOK_FLOATS;
            float v[CPL], o[CPL];
#pragma unroll
            for (int c = 0; c < CPL; c++) {
                v[c] = d[3 * ROWS + col + c];
                o[c] = 0.0f;
            }
#pragma unroll
            for (int i4 = 0; i4 < RPL / 4; i4++) {
                const float4 q4 = reinterpret_cast<const float4*>(d)[i4 * PARTS + part];
                const float4 k4 = reinterpret_cast<const float4*>(d + ROWS)[i4 * PARTS + part];
                const float4 w4 = reinterpret_cast<const float4*>(d + 2 * ROWS)[i4 * PARTS + part];
                const float q[4] = {q4.x, q4.y, q4.z, q4.w}, k[4] = {k4.x, k4.y, k4.z, k4.w}, w[4] = {w4.x, w4.y, w4.z, w4.w};
#pragma unroll
                for (int j = 0; j < 4; j++)
#pragma unroll
                    for (int c = 0; c < CPL; c++) {
                        float& st = s[i4 * 4 + j][c];
                        if (BONUS) o[c] = fmaf(q[j], st, o[c]);
                        st = fmaf(k[j], v[c], w[j] * st);
                        if (!BONUS) o[c] = fmaf(q[j], st, o[c]);
                    }
            }
#pragma unroll
            for (int off = 1; off < PARTS; off <<= 1)
#pragma unroll
                for (int c = 0; c < CPL; c++) o[c] += __shfl_xor_sync(FULL, o[c], off);
            if (part == 0) {
#pragma unroll
                for (int c = 0; c < CPL; c++) {
                    const int j = c0 + col + c;
                    if (BONUS) o[c] = fmaf(d[3 * ROWS + COLS], v[c], o[c]);
                    if (j < dv) a.o[(size_t)(t0 + t) * a.heads * dv + h * dv + j] = o[c];
                }
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < RPL; i++)
#pragma unroll
        for (int c = 0; c < CPL; c++) {
            const int r = ((i / 4) * PARTS + part) * 4 + (i & 3), j = c0 + col + c;
            if (r < dk && j < dv) S[(size_t)r * dv + j] = s[i][c];
        }
}

// RMS norm over each head's outputs, norm weight and gate: one warp per (token, head).
template <class T>
__global__ void __launch_bounds__(256) k_frecur_out(const RecurArgs a) {
    pdl_trigger();
    pdl_wait();
    const int lane = threadIdx.x & 31;
    const long long id = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (id >= (long long)a.M * a.heads) return;
    const int row = (int)(id / a.heads), h = (int)(id % a.heads), dv = a.dv;
    const float* o = a.o + (size_t)row * a.heads * dv + h * dv;
    float ss = 0.0f;
    for (int j = lane; j < dv; j += 32) ss = fmaf(o[j], o[j], ss);
    const float rs = 1.0f / sqrtf(warp_sum(ss) / (float)dv + a.eps);
    const float* gate = a.y + (size_t)row * a.ldy + a.gate_off + h * dv;
    T* out = static_cast<T*>(a.out) + (size_t)row * a.ldo + h * dv;
    for (int j = lane; j < dv; j += 32) put(out + j, o[j] * rs * a.norm[h * dv + j] * silu_fast(gate[j]));
}

template <int PARTS, int RPL, int CPL, bool BONUS>
static void launch_scan(const RecurArgs& a, cudaStream_t q) {
    constexpr int ROWS = PARTS * RPL, COLS = SC_WARPS * (32 / PARTS) * CPL;
    const size_t smem = 2 * SC_TB * (3 * ROWS + COLS + 4) * sizeof(float);
    static bool configured = false;
    if (!configured) {
        DETB_CUDA_OK(cudaFuncSetAttribute(k_frecur_scan<PARTS, RPL, CPL, BONUS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        configured = true;
    }
    launch_pdl(k_frecur_scan<PARTS, RPL, CPL, BONUS>, dim3((a.dv + COLS - 1) / COLS, a.heads), dim3(SC_THREADS), smem, q, 1, a);
}
template <bool BONUS>
static void scan(const RecurArgs& a, cudaStream_t q) {
    if (a.dk <= 32) launch_scan<4, 8, 1, BONUS>(a, q);
    else if (a.dk <= 64) launch_scan<8, 8, 1, BONUS>(a, q);
    else if (a.dk <= 128) launch_scan<8, 16, 1, BONUS>(a, q);
    else if (a.dk <= 256) launch_scan<8, 32, 1, BONUS>(a, q);
    else launch_scan<16, 32, 1, BONUS>(a, q);
}

}  // namespace detb

using namespace detb;

extern "C" {

size_t det_f_recur_scratch_bytes(int M, int heads, int dk, int dv) {
    return M > 1 ? (size_t)M * heads * (dk + dv) * sizeof(float) : 16;
}

void det_f_recur(const det_frecur_op* op, cudaStream_t st) {
    DETB_REQUIRE(op->heads > 0 && op->dk > 0 && op->dk <= 512 && op->dv > 0 && op->dv <= 4096, "recurrence: unsupported head size");
    DETB_REQUIRE(op->w2 && op->w2->N == op->heads * op->dk && op->w2->K == op->rank && op->w2->ld == round8(op->rank),
                 "recurrence: decay projection does not fit");
    if (op->M <= 0) return;
    cudaStream_t q = queue_of(st);
    RecurArgs a{};
    a.heads = op->heads; a.dk = op->dk; a.dv = op->dv; a.rank = op->rank; a.M = op->M;
    a.y = op->y; a.ldy = op->ldy;
    a.q_off = op->q_off; a.k_off = op->k_off; a.v_off = op->v_off; a.gate_off = op->gate_off; a.low_off = op->low_off;
    a.q_scale = op->q_scale; a.decay = op->decay; a.inv_tau = 1.0f / op->tau;
    a.w2 = static_cast<const bf16*>(op->w2->w); a.ldw2 = op->w2->ld;
    a.bias = op->bias; a.u = op->u; a.norm = op->norm; a.eps = op->eps;
    a.out = op->out; a.ldo = op->ldo; a.seq = op->seq;
    if (op->seq.table || op->M == 1) {
        const int vp = std::min((op->dv + 31) & ~31, RS_THREADS), ng = RS_THREADS / vp;
        const size_t smem = (3 * (size_t)op->dk + op->dv + round8(op->rank) + (size_t)ng * op->dv) * sizeof(float);
        DETB_REQUIRE(smem <= 48 * 1024, "recurrence: head or rank too large for the one-token kernel");
        dim3 grid(op->heads, op->M);
        if (op->dtype == DET_BF16) launch_pdl(k_frecur_step<bf16>, grid, dim3(RS_THREADS), smem, q, 1, a);
        else launch_pdl(k_frecur_step<float>, grid, dim3(RS_THREADS), smem, q, 1, a);
        return;
    }
    a.z = static_cast<float*>(op->scratch);
    a.o = a.z + (size_t)op->M * op->heads * op->dk;
    fdecay_launch(op->w2, op->y + op->low_off, op->ldy, op->bias, op->decay, op->tau, op->M, a.z, q);
    if (op->u) scan<true>(a, q);
    else scan<false>(a, q);
    const unsigned blocks = (unsigned)(((long long)op->M * op->heads + 7) / 8);
    if (op->dtype == DET_BF16) launch_pdl(k_frecur_out<bf16>, dim3(blocks), dim3(256), 0, q, 1, a);
    else launch_pdl(k_frecur_out<float>, dim3(blocks), dim3(256), 0, q, 1, a);
}

}  // extern "C"
