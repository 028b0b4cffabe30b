// Linear recurrences with a decay per key channel (gated linear attention and RWKV-style time mixing share one recurrence:
// include/det_b200.h, det_frecur_op).  State S[dk][dv] per head in fp32, updated in fp32.
//
//   k_frecur_step   one token per row (decode; rows may belong to different sequences): a cluster of CTAs per (head, row), each
//                   with a slab of the head's columns, computes the decays from their low-rank projection, streams the state
//                   once, exchanges the sums of squares over distributed shared memory and finishes with the head's RMS norm
//                   and gate, so a layer step is one launch.  Bound by the bytes of the states.
//   k_frecur_scan   a run of tokens of one sequence: a lane keeps RPL rows of two columns of S in registers, PARTS lanes share
//                   the columns; per-token operands arrive in shared memory by asynchronous copies, a block of tokens ahead.
//                   Bound by the issue of its multiply-adds, three per state element and token.  The decays come from
//                   k_fdecay, the norm and the gate from k_frecur_out.
#include "fops.cuh"
#include <algorithm>
#include <cooperative_groups.h>

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
constexpr int RS_THREADS = 256;

template <class T>
__global__ void __launch_bounds__(RS_THREADS) k_frecur_step(const RecurArgs a, int cs /* CTAs per head */) {
    namespace cg = cooperative_groups;
    extern __shared__ __align__(16) float rsm[];
    __shared__ float sh[32];
    __shared__ float peer_ss[8];
    const int h = blockIdx.x / cs, part_cta = blockIdx.x % cs, row = blockIdx.y, dk = a.dk, dv = a.dv, tid = threadIdx.x;
    const int per = (dv + cs - 1) / cs, j0 = part_cta * per, nj = max(0, min(dv - j0, per));   // this CTA's columns
    float* sq = rsm;                 // [dk]
    float* sk = sq + dk;             // [dk]
    float* sd = sk + dk;             // [dk] decay
    float* st = sd + dk;             // [rank rounded up to 8]
    float* sv = st + ((a.rank + 7) & ~7);   // [per]
    float* so = sv + per;            // [groups][per]
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
    for (int j = tid; j < nj; j += RS_THREADS) sv[j] = y[a.v_off + h * dv + j0 + j];
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
    // state: thread = column (rounded up to a warp) x group of rows
    float* S = slot_of(a.seq, row).s + (size_t)h * dk * dv + j0;
    const int vp = min((per + 31) & ~31, RS_THREADS), ng = RS_THREADS / vp, g = tid / vp;
    if (g < ng) {
        for (int j = tid % vp; j < nj; j += vp) {
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
            so[g * per + j] = o;
        }
    }
    __syncthreads();
    float ss = 0.0f;
    for (int j = tid; j < nj; j += RS_THREADS) {
        float o = a.u ? bonus * sv[j] : 0.0f;
        for (int x = 0; x < ng; x++) o += so[x * per + j];
        so[j] = o;
        ss = fmaf(o, o, ss);
    }
    ss = block_sum(ss, sh);
    if (cs > 1) {
        cg::cluster_group cluster = cg::this_cluster();
        if (tid < cs) *cluster.map_shared_rank(&peer_ss[part_cta], tid) = ss;
        cluster.sync();
        ss = 0.0f;
        for (int c = 0; c < cs; c++) ss += peer_ss[c];
    }
    const float rs = 1.0f / sqrtf(ss / (float)dv + a.eps);
    T* out = static_cast<T*>(a.out) + (size_t)row * a.ldo + h * dv + j0;
    for (int j = tid; j < nj; j += RS_THREADS)
        put(out + j, so[j] * rs * a.norm[h * dv + j0 + j] * silu_fast(y[a.gate_off + h * dv + j0 + j]));
}

// ------------------------------------------------------------------------------------------------------ a run of tokens
constexpr int SC_WARPS = 4, SC_THREADS = SC_WARPS * 32, SC_TB = 16, SC_CPL = 2;   // tokens per staged block, columns per lane

// Asynchronous copy of V floats to shared memory; zeros when `in` is false.
template <int V>
__device__ __forceinline__ void copy_async(float* dst, const float* src, bool in) {
    const int n = in ? V * 4 : 0;
    if constexpr (V == 4) asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_addr(dst)), "l"(src), "r"(n) : "memory");
    else asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(smem_addr(dst)), "l"(src), "r"(n) : "memory");
}

// Row r of a head, r = (i4 * PARTS + part) * 4 + j: PARTS consecutive lanes read PARTS consecutive 16-byte pieces of a staged
// vector; the dk rows are padded with zeros to PARTS * RPL.  V = 4: every operand row starts on a 16-byte boundary and dk, dv
// are multiples of 4.
template <int PARTS, int RPL, bool BONUS, int V>
__global__ void __launch_bounds__(SC_THREADS) k_frecur_scan(const RecurArgs a) {
    constexpr int ROWS = PARTS * RPL, LC = 32 / PARTS, COLS = SC_WARPS * LC * SC_CPL;
    constexpr int TOK = 3 * ROWS + COLS;                     // q | k | decay | v of a token
    extern __shared__ __align__(16) float scm[];             // [2][SC_TB][TOK]
    const int h = blockIdx.y, c0 = blockIdx.x * COLS, dk = a.dk, dv = a.dv;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, part = lane % PARTS;
    const int col = (warp * LC + lane / PARTS) * SC_CPL;     // first column of this lane inside the CTA
    pdl_trigger();
    pdl_wait();
    // a thread copies the same one or two elements of every token: pointers advance by a token
    constexpr int SLOTS = (TOK / V + SC_THREADS - 1) / SC_THREADS;
    const float* src0[SLOTS];
    int step[SLOTS];
    bool in[SLOTS];
#pragma unroll
    for (int i = 0; i < SLOTS; i++) {
        const int e = (threadIdx.x + i * SC_THREADS) * V;
        src0[i] = nullptr;
        step[i] = a.ldy;
        in[i] = false;
        if (e < 3 * ROWS) {
            const int which = e / ROWS, r = e % ROWS;
            in[i] = r < dk;
            src0[i] = which == 2 ? a.z + (size_t)h * dk : a.y + (which ? a.k_off : a.q_off) + h * dk;
            if (which == 2) step[i] = a.heads * dk;
            src0[i] += in[i] ? r : 0;
        } else if (e < TOK) {
            const int c = c0 + e - 3 * ROWS;
            in[i] = c < dv;
            src0[i] = a.y + a.v_off + h * dv + (in[i] ? c : 0);
        }
    }
    auto stage = [&](int t0, int buf) {
        const int nt = min(SC_TB, a.M - t0);
#pragma unroll
        for (int i = 0; i < SLOTS; i++) {
            if (!src0[i]) continue;
            const float* src = src0[i] + (size_t)t0 * step[i];
            float* dst = scm + buf * (SC_TB * TOK) + (threadIdx.x + i * SC_THREADS) * V;
#pragma unroll 4
            for (int t = 0; t < nt; t++, src += step[i], dst += TOK) copy_async<V>(dst, src, in[i]);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage(0, 0);
    float* S = a.seq.one.s + (size_t)h * dk * dv;
    float s[RPL][SC_CPL], u[BONUS ? RPL : 1];
#pragma unroll
    for (int i = 0; i < RPL; i++) {
        const int r = ((i / 4) * PARTS + part) * 4 + (i & 3);
        if (BONUS) u[i] = r < dk ? a.u[h * dk + r] : 0.0f;
#pragma unroll
        for (int c = 0; c < SC_CPL; c++) s[i][c] = (r < dk && c0 + col + c < dv) ? S[(size_t)r * dv + c0 + col + c] : 0.0f;
    }
    // which of its two columns a lane ends up with after the reduction below, and whether it stores it
    constexpr int HI = PARTS / 2;
    const bool up = part & HI;
    const int mine = c0 + col + (up ? 1 : 0);
    const bool stores = (part & (HI - 1)) == 0 && mine < dv;
    float* out = a.o + (size_t)h * dv + mine;
    const size_t ldo = (size_t)a.heads * dv;
    for (int t0 = 0, p = 0; t0 < a.M; t0 += SC_TB, p ^= 1) {
        if (t0 + SC_TB < a.M) {
            stage(t0 + SC_TB, p ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const int nt = min(SC_TB, a.M - t0);
        const float* d = scm + p * (SC_TB * TOK);
#pragma unroll 2
        for (int t = 0; t < nt; t++, d += TOK) {
            const float2 v2 = *reinterpret_cast<const float2*>(d + 3 * ROWS + col);
            const float v[SC_CPL] = {v2.x, v2.y};
            float o[SC_CPL] = {0.0f, 0.0f}, b = 0.0f;
#pragma unroll
            for (int i4 = 0; i4 < RPL / 4; i4++) {
                const float4 q4 = reinterpret_cast<const float4*>(d)[i4 * PARTS + part];
                const float4 k4 = reinterpret_cast<const float4*>(d + ROWS)[i4 * PARTS + part];
                const float4 w4 = reinterpret_cast<const float4*>(d + 2 * ROWS)[i4 * PARTS + part];
                const float q[4] = {q4.x, q4.y, q4.z, q4.w}, k[4] = {k4.x, k4.y, k4.z, k4.w}, w[4] = {w4.x, w4.y, w4.z, w4.w};
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    if (BONUS) b = fmaf(q[j] * u[BONUS ? i4 * 4 + j : 0], k[j], b);
#pragma unroll
                    for (int c = 0; c < SC_CPL; c++) {
                        float& st = s[i4 * 4 + j][c];
                        if (BONUS) o[c] = fmaf(q[j], st, o[c]);
                        st = fmaf(k[j], v[c], w[j] * st);
                        if (!BONUS) o[c] = fmaf(q[j], st, o[c]);
                    }
                }
            }
            if (BONUS) {
#pragma unroll
                for (int c = 0; c < SC_CPL; c++) o[c] = fmaf(b, v[c], o[c]);     // the sum over parts completes b as well
            }
            // two sums over PARTS lanes: one column per half, then fold
            float x = (up ? o[1] : o[0]) + __shfl_xor_sync(FULL, up ? o[0] : o[1], HI);
#pragma unroll
            for (int off = HI / 2; off > 0; off >>= 1) x += __shfl_xor_sync(FULL, x, off);
            if (stores) out[(size_t)(t0 + t) * ldo] = x * a.q_scale;
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < RPL; i++)
#pragma unroll
        for (int c = 0; c < SC_CPL; c++) {
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

template <int PARTS, int RPL, bool BONUS, int V>
static void launch_scan(const RecurArgs& a, cudaStream_t q) {
    constexpr int ROWS = PARTS * RPL, COLS = SC_WARPS * (32 / PARTS) * SC_CPL;
    const size_t smem = 2 * SC_TB * (3 * ROWS + COLS) * sizeof(float);
    static bool configured = false;
    if (!configured) {
        DETB_CUDA_OK(cudaFuncSetAttribute(k_frecur_scan<PARTS, RPL, BONUS, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        configured = true;
    }
    launch_plain(k_frecur_scan<PARTS, RPL, BONUS, V>, dim3((a.dv + COLS - 1) / COLS, a.heads), dim3(SC_THREADS), smem, q, a);
}
template <bool BONUS, int V>
static void scan(const RecurArgs& a, cudaStream_t q) {
    if (a.dk <= 32) launch_scan<8, 4, BONUS, V>(a, q);
    else if (a.dk <= 64) launch_scan<16, 4, BONUS, V>(a, q);
    else if (a.dk <= 128) launch_scan<16, 8, BONUS, V>(a, q);
    else if (a.dk <= 256) launch_scan<32, 8, BONUS, V>(a, q);
    else launch_scan<32, 16, BONUS, V>(a, q);
}
template <int V>
static void scan(const RecurArgs& a, cudaStream_t q) {
    if (a.u) scan<true, V>(a, q);
    else scan<false, V>(a, q);
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
        // CTAs per head: at least 32 columns each, as long as the device is not full without
        int cs = 1;
        while (cs < 8 && op->dv / (2 * cs) >= 32 && (long long)op->heads * op->M * cs < 2ll * sm_count()) cs *= 2;
        const int per = (op->dv + cs - 1) / cs, vp = std::min((per + 31) & ~31, RS_THREADS), ng = RS_THREADS / vp;
        const size_t smem = (3 * (size_t)op->dk + per + round8(op->rank) + (size_t)ng * per) * sizeof(float);
        DETB_REQUIRE(smem <= 48 * 1024, "recurrence: head or rank too large for the one-token kernel");
        dim3 grid(op->heads * cs, op->M);
        if (op->dtype == DET_BF16) launch_pdl(k_frecur_step<bf16>, grid, dim3(RS_THREADS), smem, q, cs, a, cs);
        else launch_pdl(k_frecur_step<float>, grid, dim3(RS_THREADS), smem, q, cs, a, cs);
        return;
    }
    a.z = static_cast<float*>(op->scratch);
    a.o = a.z + (size_t)op->M * op->heads * op->dk;
    fdecay_launch(op->w2, op->y + op->low_off, op->ldy, op->bias, op->decay, op->tau, op->M, a.z, q);
    auto aligned = [](const void* p, int off) { return ((reinterpret_cast<uintptr_t>(p) + 4 * (size_t)off) & 15) == 0; };
    const bool vec = op->dk % 4 == 0 && op->dv % 4 == 0 && op->ldy % 4 == 0 && aligned(op->y, op->q_off) && aligned(op->y, op->k_off) &&
                     aligned(op->y, op->v_off) && aligned(a.z, 0);
    if (vec) scan<4>(a, q);
    else scan<1>(a, q);
    const unsigned blocks = (unsigned)(((long long)op->M * op->heads + 7) / 8);
    if (op->dtype == DET_BF16) launch_pdl(k_frecur_out<bf16>, dim3(blocks), dim3(256), 0, q, 1, a);
    else launch_pdl(k_frecur_out<float>, dim3(blocks), dim3(256), 0, q, 1, a);
}

}  // extern "C"
