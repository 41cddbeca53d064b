// bf16 GEMM for many tokens on the 5th-generation tensor cores, plain or grouped by expert.
//
//   plain      Y[M][N] = epilogue(X[M][K] . W^T)
//   MOE_GLU    act[r][ff] = glu(s_r (x_r . Wg_e^T), s_r (x_r . Wu_e^T)),  r a sorted pair of expert e
//   MOE_DOWN   y[perm[r]][N] = act[r][K] . Wd_e^T
//   GLU        act[m][ff] = glu(x_m . Wg^T, x_m . Wu^T)
//
// As in the other tcgen05 kernels of the library the 128 output channels of a tile are the M
// dimension of tcgen05.mma and NTOK tokens its N dimension, one persistent CTA per SM:
//   warp 0     TMA producer: weight and activation tiles of 64 K-elements (128-byte swizzle); K past
//              the end and rows past the tensor arrive as zeros.  MOE_GLU loads a gate and an up
//              tile per stage: both multiply the one activation tile.
//   warp 1     MMA issue (one elected thread); accumulators in tensor memory, two sets, so that the
//              epilogue of a tile overlaps the MMAs of the next.  MOE_GLU keeps a gate and an up
//              accumulator per set, lane for lane, so the gated unit needs no exchange.
//   warps 2-9  epilogue: tcgen05.ld, epilogue arithmetic in f32, stores.
// The tiles of the grouped modes follow from the device-side expert offsets: every CTA lays the
// same tile list out from them (prefix sums in shared memory).  Rows of a tile past its expert's
// last pair belong to the next expert; they are multiplied and not stored.  The pair's weight
// multiplies the f32 sums, which is the sum over the weighted input without rounding it.
// Every wait on an mbarrier is bounded; on a time-out the CTA records AB2_ERR_TIMEOUT, stops
// issuing work, frees its tensor memory and returns.
#include <cuda.h>

#include <algorithm>
#include <cmath>

#include "linear_bf16.cuh"
#include "tcgen05_util.cuh"

using namespace ab2;
using namespace ab2::tc;

namespace ab2 {
int device_status_word(int **out);
int device_sm_count();
namespace {

constexpr int GB_EPI_WARPS = 8;  // two per tensor-memory quadrant: they take alternate token blocks
constexpr int GB_THREADS = 64 + GB_EPI_WARPS * 32;
constexpr int GB_A_BYTES = 128 * 128;  // 128 channels x 64 bf16
constexpr int GB_MAX_STAGES = 8;
constexpr int GB_MAX_EXPERTS = 1024;
constexpr int GB_RING_BYTES = 192 * 1024;

struct GbShared {
    uint64_t full[GB_MAX_STAGES], empty[GB_MAX_STAGES];
    uint64_t accfull[2], accempty[2];
    uint32_t tmem_base;
    int failed;
    int tile_start[GB_MAX_EXPERTS + 1];  // grouped modes: first token tile of each expert
};

template <int NTOK, int MODE>
__host__ __device__ constexpr int gb_stage_bytes() { return (MODE == LIN_MOE_GLU || MODE == LIN_GLU ? 2 : 1) * GB_A_BYTES + NTOK * 128; }
template <int NTOK, int MODE>
__host__ __device__ constexpr int gb_stages() {
    return GB_RING_BYTES / gb_stage_bytes<NTOK, MODE>() < GB_MAX_STAGES ? GB_RING_BYTES / gb_stage_bytes<NTOK, MODE>() : GB_MAX_STAGES;
}

// Walks the tile list: item -> (expert, channel tile, token tile).  Items of one CTA only grow, so
// the expert is found by moving forward.
struct GbCursor {
    int e = 0;
    __device__ __forceinline__ void find(const GbShared *sh, int it, int n_tiles, int &nt, int &mt) {
        while (it >= sh->tile_start[e + 1] * n_tiles) ++e;
        const int local = it - sh->tile_start[e] * n_tiles, m_tiles = sh->tile_start[e + 1] - sh->tile_start[e];
        nt = local / m_tiles;
        mt = local % m_tiles;
    }
};

template <int NTOK, int MODE>
__global__ void __launch_bounds__(GB_THREADS, 1)
gemm_bf16_tc_kernel(const __grid_constant__ CUtensorMap wmap, const __grid_constant__ CUtensorMap w2map,
                    const __grid_constant__ CUtensorMap xmap, LinArgs a, int *status) {
    constexpr bool DUAL = MODE == LIN_MOE_GLU || MODE == LIN_GLU, GROUPED = MODE == LIN_MOE_GLU || MODE == LIN_MOE_DOWN;
    constexpr int STAGES = gb_stages<NTOK, MODE>(), STAGE_BYTES = gb_stage_bytes<NTOK, MODE>();
    constexpr int ACC_COLS = DUAL ? 2 * NTOK : NTOK;  // tensor-memory columns of one accumulator set
    constexpr uint32_t TMEM_COLS = 2 * ACC_COLS;
    static_assert(TMEM_COLS <= 512, "two accumulator sets fit tensor memory");
    constexpr uint32_t IDESC = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(NTOK >> 3) << 17) | ((128u >> 4) << 24);
    extern __shared__ uint8_t smem_raw[];
    uint8_t *ring = (uint8_t *)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    GbShared *sh = (GbShared *)(ring + STAGES * STAGE_BYTES);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int KS = (a.K + 63) >> 6;
    const int n_tiles = (a.N + 127) >> 7;
    volatile int *failed = &sh->failed;

    if (threadIdx.x == 0) {
        for (int i = 0; i < STAGES; ++i) { bar_init(&sh->full[i], 1); bar_init(&sh->empty[i], 1); }
        for (int i = 0; i < 2; ++i) { bar_init(&sh->accfull[i], 1); bar_init(&sh->accempty[i], GB_EPI_WARPS); }
        sh->failed = 0;
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;\n" ::: "memory");
    }
    if (warp == 1) {  // tensor-memory allocation is a whole-warp operation
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(sptr(&sh->tmem_base)), "r"(TMEM_COLS));
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::);
    }
    pdl_wait();
    pdl_launch_dependents();
    const int E = GROUPED ? a.r.E : 1;
    if (warp == 0) {
        // prefix sums of the experts' token tiles, 32 experts at a time
        int base = 0;
        for (int e0 = 0; e0 < E; e0 += 32) {
            const int e = e0 + lane;
            int t = 0;
            if (e < E) {
                const int cnt = GROUPED ? a.r.offset[e + 1] - a.r.offset[e] : a.M;
                t = (cnt + NTOK - 1) / NTOK;
            }
            int inc = t;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int v = __shfl_up_sync(0xffffffffu, inc, o);
                if (lane >= o) inc += v;
            }
            if (e < E) sh->tile_start[e] = base + inc - t;
            base += __shfl_sync(0xffffffffu, inc, 31);
        }
        if (lane == 0) sh->tile_start[E] = base;
    }
    asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
    const uint32_t tmem = sh->tmem_base;
    const int items = sh->tile_start[E] * n_tiles;
    GbCursor cur;

    if (warp == 0) {
        // ---------------------------------------------------------- TMA producer
        if (lane == 0) {
            uint32_t use = 0;
            for (int it = blockIdx.x; it < items && !*failed; it += gridDim.x) {
                int nt, mt;
                cur.find(sh, it, n_tiles, nt, mt);
                const int wrow = (GROUPED ? cur.e * a.N : 0) + nt * 128;
                const int xrow = (GROUPED ? a.r.offset[cur.e] : 0) + mt * NTOK;
                for (int ks = 0; ks < KS && !*failed; ++ks, ++use) {
                    const int s = use % STAGES;
                    if (!bar_wait(&sh->empty[s], ((use / STAGES) & 1) ^ 1, failed)) break;
                    uint8_t *st = ring + s * STAGE_BYTES;
                    bar_expect_tx(&sh->full[s], STAGE_BYTES);  // what lies past a tensor arrives as zeros and counts
                    tma_load_2d(st, &wmap, ks * 64, wrow, &sh->full[s]);
                    if (DUAL) tma_load_2d(st + GB_A_BYTES, &w2map, ks * 64, wrow, &sh->full[s]);
                    tma_load_2d(st + (DUAL ? 2 : 1) * GB_A_BYTES, &xmap, ks * 64, xrow, &sh->full[s]);
                }
            }
        }
    } else if (warp == 1) {
        // ---------------------------------------------------------- MMA issue
        uint32_t use = 0, tuse = 0;
        for (int it = blockIdx.x; it < items && !*failed; it += gridDim.x, ++tuse) {
            const int ab = tuse & 1;
            if (!bar_wait(&sh->accempty[ab], ((tuse >> 1) & 1) ^ 1, failed)) break;
            asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
            const uint32_t tacc = tmem + (uint32_t)(ab * ACC_COLS);
            for (int ks = 0; ks < KS && !*failed; ++ks, ++use) {
                const int s = use % STAGES;
                if (!bar_wait(&sh->full[s], (use / STAGES) & 1, failed)) break;
                asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
                if (lane == 0) {
                    const uint32_t a0 = sptr(ring + s * STAGE_BYTES), b0 = a0 + (DUAL ? 2 : 1) * GB_A_BYTES;
#pragma unroll
                    for (int k = 0; k < 4; ++k) {
                        umma_bf16(tacc, umma_desc(a0 + k * 32), umma_desc(b0 + k * 32), IDESC, (ks | k) != 0);
                        if (DUAL) umma_bf16(tacc + NTOK, umma_desc(a0 + GB_A_BYTES + k * 32), umma_desc(b0 + k * 32), IDESC, (ks | k) != 0);
                    }
                    umma_commit(&sh->empty[s]);  // the stage is free when the MMAs retire
                }
                __syncwarp();
            }
            if (lane == 0) umma_commit(&sh->accfull[ab]);
            __syncwarp();
        }
    } else {
        // ---------------------------------------------------------- epilogue
        const int quad = warp & 3, first_block = (warp - 2) >> 2;
        uint32_t tuse = 0;
        for (int it = blockIdx.x; it < items && !*failed; it += gridDim.x, ++tuse) {
            int nt, mt;
            cur.find(sh, it, n_tiles, nt, mt);
            const int ab = tuse & 1;
            const int r0 = GROUPED ? a.r.offset[cur.e] : 0;
            const int cnt = (GROUPED ? a.r.offset[cur.e + 1] - r0 : a.M) - mt * NTOK;  // rows of this tile that exist
            const int row0 = r0 + mt * NTOK;
            if (!bar_wait(&sh->accfull[ab], (tuse >> 1) & 1, failed)) break;
            asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
            const int n = nt * 128 + quad * 32 + lane;
            constexpr int CW = DUAL ? 16 : 32;  // tokens per register block
#pragma unroll 1
            for (int c = first_block; c < NTOK / CW; c += GB_EPI_WARPS / 4) {
                __syncwarp();  // the tensor-memory load is a whole-warp operation
                if (c * CW >= cnt) break;
                const uint32_t taddr = tmem + ((uint32_t)(quad * 32) << 16) + (uint32_t)(ab * ACC_COLS + c * CW);
                uint32_t v[32];
                if (DUAL) {
#pragma unroll
                    for (int h = 0; h < 2; ++h)
                        asm volatile(
                            "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];\n"
                            : "=r"(v[16 * h]), "=r"(v[16 * h + 1]), "=r"(v[16 * h + 2]), "=r"(v[16 * h + 3]), "=r"(v[16 * h + 4]),
                              "=r"(v[16 * h + 5]), "=r"(v[16 * h + 6]), "=r"(v[16 * h + 7]), "=r"(v[16 * h + 8]), "=r"(v[16 * h + 9]),
                              "=r"(v[16 * h + 10]), "=r"(v[16 * h + 11]), "=r"(v[16 * h + 12]), "=r"(v[16 * h + 13]),
                              "=r"(v[16 * h + 14]), "=r"(v[16 * h + 15])
                            : "r"(taddr + (uint32_t)(h * NTOK)));
                } else {
                    asm volatile(
                        "tcgen05.ld.sync.aligned.32x32b.x32.b32 "
                        "{%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];\n"
                        : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]),
                          "=r"(v[8]), "=r"(v[9]), "=r"(v[10]), "=r"(v[11]), "=r"(v[12]), "=r"(v[13]), "=r"(v[14]), "=r"(v[15]),
                          "=r"(v[16]), "=r"(v[17]), "=r"(v[18]), "=r"(v[19]), "=r"(v[20]), "=r"(v[21]), "=r"(v[22]), "=r"(v[23]),
                          "=r"(v[24]), "=r"(v[25]), "=r"(v[26]), "=r"(v[27]), "=r"(v[28]), "=r"(v[29]), "=r"(v[30]), "=r"(v[31])
                        : "r"(taddr));
                }
                asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
                if (MODE == LIN_DENSE) {
                    if (n >= a.N) continue;
                    if (a.epi == LIN_F32) {
                        float *y = (float *)a.y + (row0 + c * CW) * a.ldy + n;
                        if (a.cap > 0.f) {
#pragma unroll
                            for (int j = 0; j < CW; ++j) v[j] = __float_as_uint(softcap_value(__uint_as_float(v[j]), a.cap));
                        }
#pragma unroll
                        for (int j = 0; j < CW; ++j)
                            if (c * CW + j < cnt) y[j * a.ldy] = __uint_as_float(v[j]);
                    } else {
                        __nv_bfloat16 *y = (__nv_bfloat16 *)a.y + (row0 + c * CW) * a.ldy + n;
                        const bool act = a.epi == LIN_ACT, silu = n < a.act_n;
#pragma unroll
                        for (int j = 0; j < CW; ++j) {
                            float f = __uint_as_float(v[j]);
                            if (act) {
                                const float sg = __fdividef(1.f, 1.f + __expf(-f));
                                f = silu ? f * sg : sg;
                            }
                            if (c * CW + j < cnt) y[j * a.ldy] = __float2bfloat16_rn(f);
                        }
                    }
                } else {
                    // lane j holds the pair (and its weight) of the block's token j
                    const int my_row = row0 + c * CW + lane;
                    const int my_pair = GROUPED && lane < CW && c * CW + lane < cnt ? a.r.perm[my_row] : 0;
                    const float my_score = MODE == LIN_MOE_GLU && a.scored ? a.r.score[my_pair] : 1.f;
#pragma unroll
                    for (int j = 0; j < CW; ++j) {
                        const int pair = __shfl_sync(0xffffffffu, my_pair, j);
                        const float sc = __shfl_sync(0xffffffffu, my_score, j);
                        if (c * CW + j >= cnt || n >= a.N) continue;
                        if (DUAL)
                            ((__nv_bfloat16 *)a.y)[(size_t)(row0 + c * CW + j) * a.N + n] = __float2bfloat16_rn(
                                glu_value(a.glu, sc * __uint_as_float(v[j]), sc * __uint_as_float(v[16 + j % 16]), a.limit));
                        else
                            ((float *)a.y)[(size_t)pair * a.N + n] = a.out_scale * __uint_as_float(v[j]);
                    }
                }
            }
            asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
            __syncwarp();
            if (lane == 0) bar_arrive(&sh->accempty[ab]);
        }
    }

    // ---- teardown: every warp arrives here (all waits are bounded)
    asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
    __syncthreads();
    if (threadIdx.x == 0 && sh->failed) atomicExch(status, (int)AB2_ERR_TIMEOUT);
    if (warp == 1) {
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem), "r"(TMEM_COLS));
    }
}

template <int NTOK, int MODE>
int launch_tc(const LinArgs &a, cudaStream_t s) {
    int *status = nullptr;
    int rc = device_status_word(&status);
    if (rc != AB2_OK) return rc;
    CUtensorMap wmap, w2map, xmap;
    constexpr bool GROUPED = MODE == LIN_MOE_GLU || MODE == LIN_MOE_DOWN;
    const int wrows = GROUPED ? a.N * a.r.E : a.N;
    rc = make_x_map(&wmap, a.w, wrows, a.K, 128);
    if (rc == AB2_OK) rc = make_x_map(&w2map, MODE == LIN_MOE_GLU || MODE == LIN_GLU ? a.w2 : a.w, wrows, a.K, 128);
    if (rc == AB2_OK) rc = make_x_map(&xmap, a.x, a.M, a.K, NTOK, MODE == LIN_DENSE ? a.ldx : a.K);
    if (rc != AB2_OK) return rc;
    const size_t smem = 1024 + (size_t)gb_stages<NTOK, MODE>() * gb_stage_bytes<NTOK, MODE>() + sizeof(GbShared);
    static bool configured[64] = {false};  // the attribute is per device
    int dev = 0;
    AB2_CUDA(cudaGetDevice(&dev));
    AB2_REQUIRE(dev >= 0 && dev < 64, AB2_ERR_BAD_ARG, "device index %d out of range", dev);
    if (!configured[dev]) {
        AB2_CUDA(cudaFuncSetAttribute(gemm_bf16_tc_kernel<NTOK, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        configured[dev] = true;
    }
    // at most this many tiles: every expert may leave one token tile part empty
    const long long m_tiles = (a.M + NTOK - 1) / NTOK + (GROUPED ? std::min(a.r.E, a.r.pairs) : 0);
    const int grid = (int)std::min<long long>(m_tiles * ((a.N + 127) / 128), device_sm_count());
    cudaError_t e = launch_kernel(gemm_bf16_tc_kernel<NTOK, MODE>, dim3(grid), dim3(GB_THREADS), smem, s, wmap, w2map, xmap, a, status);
    if (e != cudaSuccess) return fail(AB2_ERR_CUDA, "bf16 GEMM launch failed: %s", cudaGetErrorString(e));
    return AB2_OK;
}

}  // namespace

int gemm_bf16_tc(const LinArgs &a, int mode, cudaStream_t s) {
    // The token tile: waves of tiles over the SMs times what a tile costs, which is the rows it streams
    // through L2 - its tokens and the 128 (gate and up: 256) weight rows.  An expert's rows are counted with what
    // routing spreads around their mean.
    const int sms = device_sm_count(), n_tiles = (a.N + 127) / 128;
    const bool grouped = mode == LIN_MOE_GLU || mode == LIN_MOE_DOWN, dual = mode == LIN_MOE_GLU || mode == LIN_GLU;
    const int groups = grouped ? std::min(a.r.E, a.r.pairs) : 1;
    const double rows = !grouped ? a.M : (double)a.M / groups + std::sqrt((double)a.M / groups);
    auto cost = [&](int ntok) {
        const double tiles = std::ceil(rows / ntok) * n_tiles * groups;
        return std::ceil(tiles / sms) * (ntok + (dual ? 256 : 128));
    };
    if (mode == LIN_DENSE) {
        if (cost(256) <= cost(128) && cost(256) <= cost(64)) return launch_tc<256, LIN_DENSE>(a, s);
        return cost(128) <= cost(64) ? launch_tc<128, LIN_DENSE>(a, s) : launch_tc<64, LIN_DENSE>(a, s);
    }
    if (mode == LIN_GLU) return cost(128) <= cost(64) ? launch_tc<128, LIN_GLU>(a, s) : launch_tc<64, LIN_GLU>(a, s);
    AB2_REQUIRE(a.r.E <= GB_MAX_EXPERTS, AB2_ERR_UNSUPPORTED, "%d experts exceed the %d the grouped GEMM serves", a.r.E, GB_MAX_EXPERTS);
    if (mode == LIN_MOE_GLU) return cost(128) <= cost(64) ? launch_tc<128, LIN_MOE_GLU>(a, s) : launch_tc<64, LIN_MOE_GLU>(a, s);
    if (cost(256) <= cost(128) && cost(256) <= cost(64)) return launch_tc<256, LIN_MOE_DOWN>(a, s);
    return cost(128) <= cost(64) ? launch_tc<128, LIN_MOE_DOWN>(a, s) : launch_tc<64, LIN_MOE_DOWN>(a, s);
}

}  // namespace ab2
