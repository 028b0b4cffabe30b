// Prefill and batched-decode products of the floating-point op set on the 5th-generation tensor cores:
// tcgen05.mma kind::f16 (bfloat16 x bfloat16 -> fp32) with TMA-fed operands and TMEM accumulators.
//
// CTA tile: 128 weight rows (UMMA M, one TMEM lane per row) x TOK tokens (UMMA N: 32, 128 or 256); a stage holds 64 values
// of K of both operands (128-byte rows, SWIZZLE_128B).  Persistent: a CTA walks its tiles, tokens fastest, with two TMEM
// accumulators, so that the epilogue of one tile runs beside the loads and products of the next.  Warp 0 issues TMA, warp 1
// the MMAs, the others drain TMEM and apply the epilogue (residual add, softcap, SwiGLU of interleaved gate / up rows).
// When whole tiles would leave SMs idle in the last round, the stages of all tiles are dealt out evenly instead: a CTA may then
// begin or end inside a tile.  Such a piece goes to the library's workspace, and the CTA that arrives last at the tile adds
// its pieces in order of K, so the result does not depend on the order of arrival.
//
// Over a stack of linears (a mixture's experts) the token tiles come from a work list in device memory: a tile then is
// (entry, weight tile of the entry's linear), whole tiles are dealt round robin, and input rows are already sorted by linear.
#include "umma.cuh"
#include "fops.cuh"
#include <algorithm>

namespace detb {

constexpr int FT_ROWS = 128, FT_KE = 64;              // weight rows of a tile, elements of K per stage
constexpr int FT_A_BYTES = FT_ROWS * 128;

template <int TOK>
struct FtCfg {
    static constexpr int B_BYTES = TOK * 128;
    static constexpr int STAGE_BYTES = FT_A_BYTES + B_BYTES;
    static constexpr int STAGES = TOK == 256 ? 4 : (TOK == 128 ? 6 : 9);
    static constexpr int EPI_WARPS = TOK == 32 ? 4 : 8;
    static constexpr int THREADS = (2 + EPI_WARPS) * 32;
    static constexpr int EC = TOK * 4 / EPI_WARPS;     // token columns of an epilogue warp
    static constexpr int TMEM_COLS = 2 * TOK;
    static constexpr unsigned IDESC = (1u << 4) | (1u << 7) | (1u << 10) | ((unsigned)(TOK >> 3) << 17) | ((FT_ROWS >> 4) << 24);
    static constexpr size_t SMEM = 1024 + (size_t)STAGES * STAGE_BYTES + (2 * STAGES + 4) * 8 + 16;
};

struct FtPlan {
    int tok_tiles, wtiles, kb;            // token tiles, weight tiles, stages over the whole of K
    int tiled;                            // weights come from the tile-major copy
    int dealt;                            // stages are dealt out evenly (else whole tiles)
    int grouped;                          // tiles come from FgemmArgs.work; wtiles is per linear
    int m_rows;                           // rows of one input group in the tensor map
    float* part;                          // [CTA][2][TOK][FT_ROWS]: the piece that continues a tile, the piece that begins one
    unsigned* counters;                   // one per CTA that begins a shared tile
};

__device__ __forceinline__ void umma_bf16(unsigned tmem_d, unsigned long long da, unsigned long long db, unsigned idesc,
                                          unsigned accumulate) {
    asm volatile(
        "{\n\t.reg .pred p;\n\t"
        "setp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
        ::"r"(tmem_d), "l"(da), "l"(db), "r"(idesc), "r"(accumulate)
        : "memory");
}

// The pieces of a launch a CTA works on, one after the other.  Whole tiles are dealt round robin, tokens fastest.  Stages are
// dealt per token tile: CTA c belongs to token tile c % tok_tiles, and the CTAs of a token tile share its (weight tile, stage)
// sequence evenly, so that CTAs which read the same weights run side by side.
struct FtItem {
    TilePlace pl;
    int wt, tt, b0, nb;                   // weight tile, token tile, first stage and number of stages
    int x_row, m0, m_end;                 // first row in the tensor map; output rows of the tile
    int n_base;                           // row of W whose output is column 0
};
struct FtWalk {
    long long u, hi;                      // dealt: stage positions; else tile numbers
    int ctas, rank;                       // dealt: CTAs of this token tile and this one's place among them
};
__device__ __forceinline__ long long ft_bound(const FtPlan& p, const FtWalk& w, int rank) {
    return (long long)rank * p.wtiles * p.kb / w.ctas;
}
__device__ __forceinline__ FtWalk ft_walk(const FgemmArgs& a, const FtPlan& p) {
    FtWalk w;
    w.ctas = w.rank = 0;
    if (!p.dealt) {
        w.u = blockIdx.x;
        w.hi = (long long)p.wtiles * (p.grouped ? *a.nwork : p.tok_tiles);
        return w;
    }
    const int tt = blockIdx.x % p.tok_tiles;
    w.rank = blockIdx.x / p.tok_tiles;
    w.ctas = (gridDim.x - tt + p.tok_tiles - 1) / p.tok_tiles;
    w.u = ft_bound(p, w, w.rank);
    w.hi = ft_bound(p, w, w.rank + 1);
    return w;
}
// The rank whose run holds stage u.
__device__ __forceinline__ int ft_owner(const FtPlan& p, const FtWalk& w, long long u) {
    int c = (int)(u * w.ctas / ((long long)p.wtiles * p.kb));
    while (c + 1 < w.ctas && ft_bound(p, w, c + 1) <= u) c++;
    while (c > 0 && ft_bound(p, w, c) > u) c--;
    return c;
}
__device__ __forceinline__ bool ft_more(const FtWalk& w) { return w.u < w.hi; }
template <int TOK>
__device__ __forceinline__ FtItem ft_next(const FgemmArgs& a, const FtPlan& p, FtWalk& w) {
    FtItem it;
    it.n_base = 0;
    if (p.grouped) {
        it.tt = (int)(w.u / p.wtiles);
        const int wt = (int)(w.u - (long long)it.tt * p.wtiles);
        const int4 e = a.work[it.tt];
        it.n_base = e.x * a.group_rows;
        it.wt = e.x * p.wtiles + wt;
        it.b0 = 0;
        it.nb = p.kb;
        it.pl = TilePlace{0, it.n_base + wt * FT_ROWS, it.n_base + a.group_rows};
        it.x_row = it.m0 = e.y;
        it.m_end = e.z;
        w.u += gridDim.x;
        return it;
    }
    if (p.dealt) {
        it.wt = (int)(w.u / p.kb);
        it.tt = blockIdx.x % p.tok_tiles;
        it.b0 = (int)(w.u % p.kb);
        it.nb = (int)min((long long)(p.kb - it.b0), w.hi - w.u);
        w.u += it.nb;
    } else {
        it.wt = (int)(w.u / p.tok_tiles);
        it.tt = (int)(w.u % p.tok_tiles);
        it.b0 = 0;
        it.nb = p.kb;
        w.u += gridDim.x;
    }
    it.pl = place_tile<FT_ROWS>(a, it.wt);
    it.m0 = it.tt * TOK;
    it.m_end = a.M;
    it.x_row = a.seg_in[it.pl.seg] * p.m_rows + it.m0;
    return it;
}

// Two neighbouring tokens (columns) of one weight row: v0 at token m, v1 at token m + 1.
__device__ __forceinline__ void ft_emit2(const FgemmArgs& a, const FtItem& it, int n, int m, float v0, float v1) {
    const TilePlace& pl = it.pl;
    if (pl.n0 >= a.glu_from) {
        if (a.act == DET_FF_RELU2) {
            if (n >= pl.n_end) return;
            bf16* h = static_cast<bf16*>(a.h) + (size_t)m * a.ldh + (n - it.n_base - a.glu_from);
            if (m < it.m_end) put(h, relu_squared(v0));
            if (m + 1 < it.m_end) put(h + a.ldh, relu_squared(v1));
            return;
        }
        // lanes 2i / 2i + 1 hold gate / up: the even lane takes token m, the odd one token m + 1
        const bool odd = threadIdx.x & 1;
        const float got = __shfl_xor_sync(FULL, odd ? v0 : v1, 1);
        const float g = odd ? got : v0, u = odd ? v1 : got;
        const int mm = m + (odd ? 1 : 0);
        if (n < pl.n_end && mm < it.m_end)
            put(static_cast<bf16*>(a.h) + (size_t)mm * a.ldh + (n - a.glu_from) / 2, gate_pair(a.act, g, u));
        return;
    }
    if (n >= pl.n_end) return;
    if (a.bias) {
        const float b = a.bias[n];
        v0 += b;
        v1 += b;
    }
    if (a.softcap > 0.0f) {
        v0 = a.softcap * tanhf(v0 / a.softcap);
        v1 = a.softcap * tanhf(v1 / a.softcap);
    }
    const size_t at = (size_t)m * a.ldy + n - it.n_base;
    if (a.yb) {
        if (m < it.m_end) put(a.yb + at, v0);
        if (m + 1 < it.m_end) put(a.yb + at + a.ldy, v1);
    } else if (a.accumulate) {
        if (m < it.m_end) a.y[at] += v0;
        if (m + 1 < it.m_end) a.y[at + a.ldy] += v1;
    } else {
        if (m < it.m_end) a.y[at] = v0;
        if (m + 1 < it.m_end) a.y[at + a.ldy] = v1;
    }
}

template <int TOK>
__global__ void __launch_bounds__(FtCfg<TOK>::THREADS, 1)
k_fgemm_tc(const __grid_constant__ CUtensorMap map_w, const __grid_constant__ CUtensorMap map_x, const FgemmArgs a, const FtPlan p) {
    using Cfg = FtCfg<TOK>;
    constexpr int STAGES = Cfg::STAGES;
    extern __shared__ __align__(1024) uint8_t ft_raw[];
    uint8_t* stages = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(ft_raw) + 1023) & ~(uintptr_t)1023);
    unsigned long long* full = reinterpret_cast<unsigned long long*>(stages + (size_t)STAGES * Cfg::STAGE_BYTES);
    unsigned long long* empty = full + STAGES;
    unsigned long long* tfull = empty + STAGES;      // [2] accumulator complete
    unsigned long long* tempty = tfull + 2;          // [2] accumulator drained
    unsigned* tmem_slot = reinterpret_cast<unsigned*>(tempty + 2);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long wl = wait_limit(a.error_flag);
    pdl_trigger();
    if (threadIdx.x == 0) {
        for (int s = 0; s < STAGES; s++) {
            mbar_init(&full[s], 1);
            mbar_init(&empty[s], 1);
        }
        for (int b = 0; b < 2; b++) {
            mbar_init(&tfull[b], 1);
            mbar_init(&tempty[b], Cfg::EPI_WARPS);
        }
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) tmem_alloc(tmem_slot, Cfg::TMEM_COLS);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const unsigned tmem = *tmem_slot;
    if (p.grouped) pdl_wait();                       // the work list is the previous kernels' result
    FtWalk walk = ft_walk(a, p);
    bool ok = true;

    if (warp == 0) {
        if (lane == 0) {
            // the weight boxes of the first stages do not depend on the previous kernel
            FtWalk ahead = walk;
            const bool any = ft_more(walk);          // a short work list leaves CTAs without a tile
            FtItem first{};
            if (any) first = ft_next<TOK>(a, p, ahead);
            auto load_w = [&](uint8_t* st, const FtItem& it, int b, unsigned long long* bar) {
                if (p.tiled) tma_load_2d(st, &map_w, 0, (it.wt * p.kb + b) * FT_ROWS, bar);
                else tma_load_2d(st, &map_w, b * FT_KE, it.pl.n0, bar);
            };
            const int lead = min(first.nb, STAGES);
            for (int l = 0; l < lead; l++) {
                mbar_expect_tx(&full[l], Cfg::STAGE_BYTES);
                load_w(stages + (size_t)l * Cfg::STAGE_BYTES, first, first.b0 + l, &full[l]);
            }
            pdl_wait();
            unsigned c = 0;                          // stages issued so far
            while (ft_more(walk) && ok) {
                const FtItem it = ft_next<TOK>(a, p, walk);
                for (int l = 0; l < it.nb; l++, c++) {
                    const int s = c % STAGES;
                    uint8_t* st = stages + (size_t)s * Cfg::STAGE_BYTES;
                    if (c >= (unsigned)lead) {
                        ok = mbar_wait(&empty[s], ((c / STAGES) & 1u) ^ 1u, wl);
                        if (!ok) break;
                        mbar_expect_tx(&full[s], Cfg::STAGE_BYTES);
                        load_w(st, it, it.b0 + l, &full[s]);
                    }
                    tma_load_2d(st + FT_A_BYTES, &map_x, (it.b0 + l) * FT_KE, it.x_row, &full[s]);
                }
            }
            if (!ok) {
                atomicExch(a.error_flag, DETB_ERR_WAIT_EXPIRED);
                for (unsigned k = 1; k <= (unsigned)STAGES && k <= c; k++)
                    (void)mbar_wait(&full[(c - k) % STAGES], ((c - k) / STAGES) & 1u, wl);
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            unsigned c = 0, t = 0;
            for (; ft_more(walk) && ok; t++) {
                const FtItem it = ft_next<TOK>(a, p, walk);
                const unsigned b = t & 1u;
                ok = mbar_wait(&tempty[b], ((t >> 1) & 1u) ^ 1u, wl);
                if (!ok) break;
                tc_fence_after();
                for (int l = 0; l < it.nb; l++, c++) {
                    const int s = c % STAGES;
                    ok = mbar_wait(&full[s], (c / STAGES) & 1u, wl);
                    if (!ok) break;
                    tc_fence_after();
                    const uint8_t* st = stages + (size_t)s * Cfg::STAGE_BYTES;
                    const unsigned long long da = umma_desc(st), db = umma_desc(st + FT_A_BYTES);
#pragma unroll
                    for (int k = 0; k < 4; k++) umma_bf16(tmem + b * TOK, da + 2 * k, db + 2 * k, Cfg::IDESC, (l | k) ? 1u : 0u);
                    umma_commit(&empty[s]);
                }
                if (ok) umma_commit(&tfull[b]);
            }
            if (!ok) atomicExch(a.error_flag, DETB_ERR_WAIT_EXPIRED);
        }
    } else {
        const int q = warp & 3, col0 = ((warp - 2) >> 2) * Cfg::EC, et = threadIdx.x - 64;
        pdl_wait();
        unsigned t = 0;
        constexpr size_t PIECE = (size_t)TOK * FT_ROWS;
        for (; ft_more(walk) && ok; t++) {
            const FtItem it = ft_next<TOK>(a, p, walk);
            const unsigned b = t & 1u;
            ok = mbar_wait(&tfull[b], (t >> 1) & 1u, wl);
            if (!ok) break;
            tc_fence_after();
            const int n = it.pl.n0 + q * 32 + lane, m0 = it.m0 + col0;
            const unsigned taddr = tmem + ((unsigned)(q * 32) << 16) + b * TOK + col0;
            const bool whole = it.nb == p.kb;
            float* mine = p.part + ((size_t)blockIdx.x * 2 + (it.b0 == 0 ? 1 : 0)) * PIECE + (size_t)col0 * FT_ROWS + q * 32 + lane;
            for (int c = 0; c < Cfg::EC; c += 32) {
                int r[32];
                tmem_ld(taddr + c, r);
                tmem_wait_ld();
                if (c + 32 >= Cfg::EC) {
                    tc_fence_before();
                    __syncwarp();
                    if (lane == 0) mbar_arrive(&tempty[b]);
                }
                if (m0 + c >= it.m_end) continue;
                if (whole) {
#pragma unroll
                    for (int j = 0; j < 32; j += 2)
                        ft_emit2(a, it, n, m0 + c + j, __int_as_float(r[j]), __int_as_float(r[j + 1]));
                } else {
#pragma unroll
                    for (int j = 0; j < 32; j++) mine[(size_t)(c + j) * FT_ROWS] = __int_as_float(r[j]);
                }
            }
            if (whole) continue;
            // a piece: the tile's CTAs meet at a counter; the last one adds the pieces
            __shared__ unsigned last_cta;
            const long long u0 = (long long)it.wt * p.kb;
            const int first = ft_owner(p, walk, u0), end = ft_owner(p, walk, u0 + p.kb - 1);   // ranks; CTA = rank * tok_tiles + tt
            unsigned* counter = p.counters + first * p.tok_tiles + it.tt;
            __threadfence();
            asm volatile("bar.sync 1, %0;" ::"n"(Cfg::EPI_WARPS * 32) : "memory");
            if (et == 0) last_cta = atomicAdd(counter, 1u) == (unsigned)(end - first);
            asm volatile("bar.sync 1, %0;" ::"n"(Cfg::EPI_WARPS * 32) : "memory");
            if (last_cta) {
                __threadfence();
                if (et == 0) *counter = 0;
                const float* all = p.part + (size_t)col0 * FT_ROWS + q * 32 + lane;
                for (int c = 0; c < Cfg::EC && m0 + c < a.M; c += 32) {
                    float v[32];
#pragma unroll
                    for (int j = 0; j < 32; j++) v[j] = 0.0f;
                    for (int s = first; s <= end; s++) {
                        const float* piece = all + ((size_t)(s * p.tok_tiles + it.tt) * 2 + (s == first ? 1 : 0)) * PIECE + (size_t)c * FT_ROWS;
#pragma unroll
                        for (int j = 0; j < 32; j++) v[j] += __ldcg(piece + (size_t)j * FT_ROWS);
                    }
#pragma unroll
                    for (int j = 0; j < 32; j += 2) ft_emit2(a, it, n, m0 + c + j, v[j], v[j + 1]);
                }
            }
            asm volatile("bar.sync 1, %0;" ::"n"(Cfg::EPI_WARPS * 32) : "memory");   // last_cta is read before it is written again
        }
        if (!ok && lane == 0) atomicExch(a.error_flag, DETB_ERR_WAIT_EXPIRED);
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) tmem_dealloc(tmem, Cfg::TMEM_COLS);
}

// A [rows][ld] bfloat16 matrix as a map with 64-column boxes (128 bytes, swizzled), zero fill outside.
static CUtensorMap bf16_map(const void* base, size_t rows, int ld, int box_rows) {
    CUtensorMap map;
    const cuuint64_t dims[2] = {(cuuint64_t)ld, (cuuint64_t)rows};
    const cuuint64_t strides[1] = {(cuuint64_t)ld * 2};
    const cuuint32_t box[2] = {(cuuint32_t)FT_KE, (cuuint32_t)box_rows};
    const cuuint32_t estr[2] = {1, 1};
    const CUresult r = encode_fn()(&map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr,
                                   CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                                   CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    DETB_REQUIRE(r == CUDA_SUCCESS, "cuTensorMapEncodeTiled failed");
    return map;
}

template <int TOK>
static void configure() {
    static bool configured = false;
    if (configured) return;
    DETB_CUDA_OK(cudaFuncSetAttribute(k_fgemm_tc<TOK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)FtCfg<TOK>::SMEM));
    configured = true;
}
// a.M: rows of x
template <int TOK>
static void launch_grouped(const FgemmArgs& a, cudaStream_t q) {
    using Cfg = FtCfg<TOK>;
    FtPlan p{};
    p.grouped = 1;
    p.kb = (a.K + FT_KE - 1) / FT_KE;
    p.wtiles = (a.group_rows + FT_ROWS - 1) / FT_ROWS;
    p.tiled = a.wt != nullptr;
    DETB_REQUIRE(a.ldw == round8(a.K), "linear: weight rows must be padded to 8 elements");
    const CUtensorMap map_w = p.tiled ? bf16_map(a.wt, (size_t)a.groups * p.wtiles * p.kb * FT_ROWS, FT_KE, FT_ROWS)
                                      : bf16_map(a.w, a.N, a.ldw, FT_ROWS);
    const CUtensorMap map_x = bf16_map(a.x, a.M, a.ldx, TOK);
    configure<TOK>();
    const int grid = (int)std::min<long long>(sm_count(), (long long)a.max_work * p.wtiles);
    launch_pdl(k_fgemm_tc<TOK>, dim3(grid), dim3(Cfg::THREADS), Cfg::SMEM, q, 1, map_w, map_x, a, p);
}

template <int TOK>
static void launch_tok(FgemmArgs a, cudaStream_t q) {
    using Cfg = FtCfg<TOK>;
    plan_tiles(a, FT_ROWS);
    if (a.group_rows) {
        launch_grouped<TOK>(a, q);
        return;
    }
    int groups = 1;
    for (int s = 0; s < a.nseg; s++) groups = std::max(groups, a.seg_in[s] + 1);
    FtPlan p{};
    p.tok_tiles = (a.M + TOK - 1) / TOK;
    p.kb = (a.K + FT_KE - 1) / FT_KE;
    p.wtiles = a.tile0[a.nseg];
    const int sms = sm_count(), tiles = p.wtiles * p.tok_tiles;
    int grid = std::min(tiles, sms);
    if (!(float_flags() & 4)) {
        // deal out stages when whole tiles keep less than 80 % of the SM-rounds busy, and a share is worth the hand-over
        const long long units = (long long)tiles * p.kb;
        const int rounds = (tiles + sms - 1) / sms, share = TOK == 32 ? 6 : 16;
        const int want = (int)std::min<long long>(sms, units / share);
        size_t bytes = 0;
        int ncnt = 0;
        p.part = fsplit_workspace(&bytes);
        p.counters = fsplit_counters(&ncnt);
        if (tiles < 0.8 * rounds * sms && want >= grid && want >= 2 * p.tok_tiles && want <= ncnt &&
            (size_t)want * 2 * TOK * FT_ROWS * sizeof(float) <= bytes) {
            p.dealt = 1;
            grid = want;
        }
    }
    // input groups lie gstride elements apart; a map row is one row of the buffer
    DETB_REQUIRE(groups == 1 || a.gstride % a.ldx == 0, "input groups must be whole rows apart");
    p.m_rows = groups == 1 ? 0 : (int)(a.gstride / a.ldx);
    const size_t x_rows = (size_t)(groups - 1) * p.m_rows + a.M;
    DETB_REQUIRE(a.ldw == round8(a.K), "linear: weight rows must be padded to 8 elements");
    p.tiled = a.wt != nullptr;
    const CUtensorMap map_w = p.tiled ? bf16_map(a.wt, (size_t)p.wtiles * p.kb * FT_ROWS, FT_KE, FT_ROWS) : bf16_map(a.w, a.N, a.ldw, FT_ROWS);
    const CUtensorMap map_x = bf16_map(a.x, x_rows, a.ldx, TOK);
    configure<TOK>();
    launch_pdl(k_fgemm_tc<TOK>, dim3(grid), dim3(Cfg::THREADS), Cfg::SMEM, q, 1, map_w, map_x, a, p);
}

// One 16-byte piece (8 values of a row) per thread.
__global__ void k_flinear_tile(const FgemmArgs a, int kb, bf16* __restrict__ dst) {
    const long long id = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    const int per_tile = kb * FT_ROWS * (FT_KE / 8);
    if (id >= (long long)a.tile0[a.nseg] * per_tile) return;
    const int t = (int)(id / per_tile), i = (int)(id % per_tile);
    const int b = i / (FT_ROWS * 8), r = i / 8 % FT_ROWS, k = b * FT_KE + (i & 7) * 8;
    TilePlace pl;
    if (a.group_rows) {
        const int per = (a.group_rows + FT_ROWS - 1) / FT_ROWS, e = t / per;
        pl = TilePlace{0, e * a.group_rows + (t - e * per) * FT_ROWS, (e + 1) * a.group_rows};
    } else {
        pl = place_tile<FT_ROWS>(a, t);
    }
    uint4 v = make_uint4(0, 0, 0, 0);
    if (pl.n0 + r < pl.n_end && k < a.ldw) v = *reinterpret_cast<const uint4*>(a.w + (size_t)(pl.n0 + r) * a.ldw + k);
    reinterpret_cast<uint4*>(dst)[id] = v;
}

void fgemm_tc_launch(FgemmArgs a, cudaStream_t q) {
    if (a.M <= 32) launch_tok<32>(a, q);
    else if (a.M <= 128) launch_tok<128>(a, q);
    else launch_tok<256>(a, q);
}
void fgemm_tc_group_launch(FgemmArgs a, int tok, cudaStream_t q) {
    if (tok == 32) launch_tok<32>(a, q);
    else launch_tok<128>(a, q);
}

}  // namespace detb

using namespace detb;

static FgemmArgs tile_args(int K, int nseg, const int* seg_end) {
    DETB_REQUIRE(K > 0 && nseg >= 1 && nseg <= 8, "linear: bad segments");
    FgemmArgs a{};
    a.K = K;
    a.nseg = nseg;
    for (int i = 0; i < nseg; i++) a.seg_end[i] = seg_end[i];
    plan_tiles(a, FT_ROWS);
    return a;
}

static void tile_rows(const FgemmArgs& a, int nseg, void* dst, cudaStream_t st) {
    const int kb = (a.K + FT_KE - 1) / FT_KE;
    const long long n = (long long)a.tile0[nseg] * kb * FT_ROWS * (FT_KE / 8);
    k_flinear_tile<<<(unsigned)((n + 255) / 256), 256, 0, queue_of(st)>>>(a, kb, static_cast<bf16*>(dst));
    DETB_CUDA_OK(cudaGetLastError());
}

extern "C" {

size_t det_f_linear_tile_bytes(int K, int nseg, const int* seg_end) {
    return (size_t)tile_args(K, nseg, seg_end).tile0[nseg] * ((K + FT_KE - 1) / FT_KE) * FT_A_BYTES;
}
void det_f_linear_tile(const det_flinear* src, int nseg, const int* seg_end, void* dst, cudaStream_t st) {
    FgemmArgs a = tile_args(src->K, nseg, seg_end);
    DETB_REQUIRE(seg_end[nseg - 1] == src->N && src->ld % 8 == 0, "linear: bad segments");
    a.w = static_cast<const bf16*>(src->w);
    a.N = src->N;
    a.ldw = src->ld;
    tile_rows(a, nseg, dst, st);
}
size_t det_f_linear_tile_groups_bytes(int K, int groups, int rows) {
    return (size_t)groups * ((rows + FT_ROWS - 1) / FT_ROWS) * ((K + FT_KE - 1) / FT_KE) * FT_A_BYTES;
}
void det_f_linear_tile_groups(const det_flinear* src, int groups, void* dst, cudaStream_t st) {
    DETB_REQUIRE(groups > 0 && src->N % groups == 0 && src->ld % 8 == 0, "linear: bad groups");
    FgemmArgs a = tile_args(src->K, 1, &src->N);
    a.group_rows = src->N / groups;
    a.tile0[1] = groups * ((a.group_rows + FT_ROWS - 1) / FT_ROWS);
    a.w = static_cast<const bf16*>(src->w);
    a.N = src->N;
    a.ldw = src->ld;
    tile_rows(a, 1, dst, st);
}

}  // extern "C"
