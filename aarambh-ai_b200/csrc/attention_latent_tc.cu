// Attention in the latent space in bf16 on the 5th-generation tensor cores: the rows are 32 (token, head)
// pairs of one sequence, the keys the cached rows [latent | rotated part] and the values the latents, so one
// tile in shared memory is the operand of both products.
//
//   S^T[64 keys][32 rows]    = K . Q^T           A: the tile, K-major;  B: the queries, K-major
//   O^T[rank][32 hi | 32 lo] += C^T . [P_hi P_lo] A: the same tile, M-major; B: the weights, N-major
//
// The softmax weights enter as two bf16 terms, the rounded weight and what rounding left, side by side as 64
// columns whose sums are added at the end: they carry about 16 significant bits.
//
//   warp 0     TMA producer: tiles of 64 keys as boxes of 64 dimensions (128-byte swizzle); what the row
//              does not have arrives as zeros.  Keys of earlier steps are requested before the dependency wait.
//   warp 1     MMA issue: the scores of the next tile go ahead of the sums of this one
//   warps 2-5  softmax: a lane holds one key and 16 rows (the upper half warp takes the upper rows), weights
//              relative to a maximum per row that moves only when a score exceeds it by 2^8 (then the
//              sums in tensor memory are rescaled), and the result at the end
// The keys are cut into nsplit runs (grid x); latent_merge_kernel adds the runs.
// Every wait on an mbarrier is bounded; on a time-out the CTA records AB2_ERR_TIMEOUT, stops issuing
// work, frees its tensor memory and returns.
#include <algorithm>

#include "stack.cuh"
#include "tcgen05_util.cuh"

using namespace ab2;
using namespace ab2::tc;

namespace ab2 {
int device_status_word(int **out);
int device_sm_count();
namespace {

constexpr int LT_KEYS = 64, LT_ROWS = LATENT_ROWS, LT_THREADS = 192, LT_MAX_STAGES = 4;
constexpr int LT_KBOX = LT_KEYS * 128, LT_QBOX = LT_ROWS * 128, LT_PBUF = LT_KEYS * 128;
constexpr int LT_MAX_BOXES = 9, LT_MAX_RANK = 512;
constexpr float LT_SLACK = 8.f;  // powers of two a score may exceed the row's maximum by

struct LtShared {
    uint64_t full[LT_MAX_STAGES], empty[LT_MAX_STAGES], qfull;
    uint64_t sfull[2], pfull[2], odone[2];
    uint32_t tmem_base;
    int failed;
    int limit[LT_ROWS];       // last position a row sees
    float red[4][LT_ROWS], top[LT_ROWS], corr[LT_ROWS];
};

struct LtArgs {
    LatentArgs a;
    __nv_bfloat16 *ox;
    int boxes, stage_boxes, mtiles, stages;  // boxes of a cache row, boxes a stage has room for, tiles of 128 latent dimensions
    uint32_t tmem_cols;
};

// M- or N-major operand, 128-byte swizzle: 64 elements of M per row of K, 8 rows a group of 1024 bytes,
// the next 64 elements `lbo` bytes further.
__device__ __forceinline__ uint64_t umma_desc_mn(uint32_t saddr, uint32_t lbo) {
    uint64_t d = 0;
    d |= (uint64_t)((saddr >> 4) & 0x3FFF);
    d |= (uint64_t)(lbo >> 4) << 16;
    d |= (uint64_t)(1024 >> 4) << 32;
    d |= (uint64_t)1 << 46;
    d |= (uint64_t)2 << 61;
    return d;
}
// Barrier of the four softmax warps; returns whether any of them passed true.
__device__ __forceinline__ bool softmax_any(bool p) {
    uint32_t r;
    asm volatile("{\n .reg .pred p, q;\n setp.ne.b32 p, %1, 0;\n barrier.cta.red.or.pred q, 1, 128, p;\n selp.u32 %0, 1, 0, q;\n}\n" : "=r"(r) : "r"((uint32_t)p) : "memory");
    return r != 0;
}
#define LT_REGS32(v) \
    "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]), "=r"(v[8]), "=r"(v[9]), "=r"(v[10]), "=r"(v[11]), \
    "=r"(v[12]), "=r"(v[13]), "=r"(v[14]), "=r"(v[15]), "=r"(v[16]), "=r"(v[17]), "=r"(v[18]), "=r"(v[19]), "=r"(v[20]), "=r"(v[21]), "=r"(v[22]), \
    "=r"(v[23]), "=r"(v[24]), "=r"(v[25]), "=r"(v[26]), "=r"(v[27]), "=r"(v[28]), "=r"(v[29]), "=r"(v[30]), "=r"(v[31])
#define LT_REGS32_IO(v) \
    "+r"(v[0]), "+r"(v[1]), "+r"(v[2]), "+r"(v[3]), "+r"(v[4]), "+r"(v[5]), "+r"(v[6]), "+r"(v[7]), "+r"(v[8]), "+r"(v[9]), "+r"(v[10]), "+r"(v[11]), \
    "+r"(v[12]), "+r"(v[13]), "+r"(v[14]), "+r"(v[15]), "+r"(v[16]), "+r"(v[17]), "+r"(v[18]), "+r"(v[19]), "+r"(v[20]), "+r"(v[21]), "+r"(v[22]), \
    "+r"(v[23]), "+r"(v[24]), "+r"(v[25]), "+r"(v[26]), "+r"(v[27]), "+r"(v[28]), "+r"(v[29]), "+r"(v[30]), "+r"(v[31])
__device__ __forceinline__ void tmem_ld32(uint32_t (&v)[32], uint32_t addr) {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x32.b32 "
        "{%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];\n"
        : LT_REGS32(v) : "r"(addr));
}
__device__ __forceinline__ void tmem_st32(uint32_t addr, const uint32_t (&v)[32]) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x32.b32 [%32], "
        "{%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31};\n" ::
            "r"(v[0]), "r"(v[1]), "r"(v[2]), "r"(v[3]), "r"(v[4]), "r"(v[5]), "r"(v[6]), "r"(v[7]), "r"(v[8]), "r"(v[9]), "r"(v[10]), "r"(v[11]),
        "r"(v[12]), "r"(v[13]), "r"(v[14]), "r"(v[15]), "r"(v[16]), "r"(v[17]), "r"(v[18]), "r"(v[19]), "r"(v[20]), "r"(v[21]), "r"(v[22]), "r"(v[23]),
        "r"(v[24]), "r"(v[25]), "r"(v[26]), "r"(v[27]), "r"(v[28]), "r"(v[29]), "r"(v[30]), "r"(v[31]), "r"(addr) : "memory");
}
// The registers pass through the wait, so that nothing computed from them can move ahead of it.
__device__ __forceinline__ void tmem_wait_ld(uint32_t (&v)[32]) {
    asm volatile("tcgen05.wait::ld.sync.aligned;\n" : LT_REGS32_IO(v)::"memory");
}

// Reduces 16 values per lane over the half warp's 16 lanes: lane L ends with the result of its value L & 15.
template <class Op>
__device__ __forceinline__ float reduce_transposed(float (&v)[16], int lane, Op op) {
#pragma unroll
    for (int w = 8; w > 0; w >>= 1) {
        const bool up = lane & w;
#pragma unroll
        for (int j = 0; j < w; ++j) {
            const float send = up ? v[j] : v[j + w], keep = up ? v[j + w] : v[j];
            v[j] = op(keep, __shfl_xor_sync(0xffffffffu, send, w));
        }
    }
    return v[0];
}

__global__ void __launch_bounds__(LT_THREADS, 1)
latent_tc_kernel(const __grid_constant__ CUtensorMap kmap, const __grid_constant__ CUtensorMap qmap, LtArgs p, int *status) {
    extern __shared__ uint8_t smem_raw[];
    uint8_t *ring = (uint8_t *)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    const LatentArgs &a = p.a;
    const int stage_bytes = p.stage_boxes * LT_KBOX;
    uint8_t *qbuf = ring + p.stages * stage_bytes, *pbuf = qbuf + p.boxes * LT_QBOX;
    LtShared *sh = (LtShared *)(pbuf + 2 * LT_PBUF);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    volatile int *failed = &sh->failed;

    const int rrow = blockIdx.z, row = kv_row(a.kv, a.row0, rrow), len = a.kv.lens[row];  // committed by earlier steps
    const int rows = a.S * a.H, r0 = blockIdx.y * LT_ROWS;
    const int n = len + min(rows - 1, r0 + LT_ROWS - 1) / a.H + 1;
    const int per = ((n + a.nsplit - 1) / a.nsplit + LT_KEYS - 1) / LT_KEYS * LT_KEYS;
    const int j0 = (int)blockIdx.x * per, j1 = min(n, j0 + per), tiles = j1 > j0 ? (j1 - j0 + LT_KEYS - 1) / LT_KEYS : 0;

    if (threadIdx.x == 0) {
        for (int i = 0; i < p.stages; ++i) { bar_init(&sh->full[i], 1); bar_init(&sh->empty[i], 1); }
        bar_init(&sh->qfull, 1);
        for (int i = 0; i < 2; ++i) { bar_init(&sh->sfull[i], 1); bar_init(&sh->pfull[i], 4); bar_init(&sh->odone[i], 1); }
        sh->failed = 0;
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;\n" ::: "memory");
    }
    if (threadIdx.x >= 64 && threadIdx.x < 64 + LT_ROWS) sh->limit[threadIdx.x - 64] = len + (r0 + (int)threadIdx.x - 64) / a.H;
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(sptr(&sh->tmem_base)), "r"(p.tmem_cols));
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::);
    }
    asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
    const uint32_t tmem = sh->tmem_base, tmem_o = tmem + 64;  // two score buffers of 32 columns, then 64 per tile of latent dimensions

    if (warp == 0) {
        // ---------------------------------------------------------- TMA producer
        if (lane == 0) {
            bool waited = false;
            auto start = [&]() {
                pdl_wait();
                pdl_launch_dependents();
                waited = true;
                if (tiles == 0) return;
                bar_expect_tx(&sh->qfull, (uint32_t)(p.boxes * LT_QBOX));
                for (int b = 0; b < p.boxes; ++b) tma_load_2d(qbuf + b * LT_QBOX, &qmap, b * 64, rrow * rows + r0, &sh->qfull);
            };
            for (int i = 0; i < tiles && !*failed; ++i) {
                const int s = i % p.stages, key = j0 + i * LT_KEYS;
                if (!waited && (i >= p.stages || key + LT_KEYS > len)) start();  // the tile has keys of this step
                if (!bar_wait(&sh->empty[s], ((i / p.stages) & 1) ^ 1, failed)) break;
                uint8_t *st = ring + s * stage_bytes;
                bar_expect_tx(&sh->full[s], (uint32_t)(p.boxes * LT_KBOX));
                for (int b = 0; b < p.boxes; ++b) tma_load_2d(st + b * LT_KBOX, &kmap, b * 64, row * a.kv.l.cap + key, &sh->full[s]);
            }
            if (!waited) start();
        }
    } else if (warp == 1) {
        // ---------------------------------------------------------- MMA issue
        constexpr uint32_t IDESC = (1u << 4) | (1u << 7) | (1u << 10);
        constexpr uint32_t IDESC_S = IDESC | ((uint32_t)(LT_ROWS >> 3) << 17) | ((64u >> 4) << 24);
        constexpr uint32_t IDESC_O = IDESC | (1u << 15) | (1u << 16) | ((uint32_t)((2 * LT_ROWS) >> 3) << 17) | ((128u >> 4) << 24);
        auto scores = [&](int i) {
            const int s = i % p.stages;
            if (!bar_wait(&sh->full[s], (i / p.stages) & 1, failed)) return false;
            asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
            if (lane == 0) {
                const uint32_t a0 = sptr(ring + s * stage_bytes), b0 = sptr(qbuf), d = tmem + (uint32_t)((i & 1) * LT_ROWS);
                for (int b = 0; b < p.boxes; ++b)
#pragma unroll
                    for (int k = 0; k < 4; ++k)
                        umma_bf16(d, umma_desc(a0 + b * LT_KBOX + k * 32), umma_desc(b0 + b * LT_QBOX + k * 32), IDESC_S, (b | k) != 0);
                umma_commit(&sh->sfull[i & 1]);
            }
            __syncwarp();
            return true;
        };
        bool ok = tiles > 0 && bar_wait(&sh->qfull, 0, failed) && scores(0);
        for (int i = 0; ok && i < tiles; ++i) {
            if (i + 1 < tiles) ok = scores(i + 1);
            if (!ok || !bar_wait(&sh->pfull[i & 1], (i >> 1) & 1, failed)) break;
            asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
            if (lane == 0) {
                const uint32_t a0 = sptr(ring + (i % p.stages) * stage_bytes), b0 = sptr(pbuf + (i & 1) * LT_PBUF);
                for (int m = 0; m < p.mtiles; ++m)
#pragma unroll
                    for (int k = 0; k < LT_KEYS / 16; ++k)
                        umma_bf16(tmem_o + (uint32_t)(m * 2 * LT_ROWS), umma_desc_mn(a0 + 2 * m * LT_KBOX + k * 2048, LT_KBOX),
                                  umma_desc_mn(b0 + k * 2048, LT_PBUF), IDESC_O, (i | k) != 0);
                umma_commit(&sh->empty[i % p.stages]);
                umma_commit(&sh->odone[i & 1]);
            }
            __syncwarp();
        }
    } else {
        // ---------------------------------------------------------- softmax
        const int quad = warp & 3, half = lane >> 4, key_in = quad * 16 + (lane & 15);
        const uint32_t quad_addr = (uint32_t)(quad * 32) << 16;
        const float sl = a.scale * 1.44269504088896341f;  // scores in powers of two
        float top[16], sum[16];
#pragma unroll
        for (int j = 0; j < 16; ++j) { top[j] = -1e30f; sum[j] = 0.f; }
        const int limit_lo = sh->limit[0];  // limits grow with the row
        pdl_wait();
        bool ok = true;
        for (int i = 0; i < tiles; ++i) {
            const int b = i & 1, key = j0 + i * LT_KEYS + key_in;
            ok = bar_wait(&sh->sfull[b], (i >> 1) & 1, failed);
            asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
            __syncwarp();
            uint32_t v[32];
            tmem_ld32(v, tmem + quad_addr + (uint32_t)(b * LT_ROWS));
            tmem_wait_ld(v);
            float s[16];
#pragma unroll
            for (int j = 0; j < 16; ++j) {  // the upper half warp takes rows 16..31 of the lower half's keys
                const float hi = __shfl_sync(0xffffffffu, __uint_as_float(v[16 + j]), lane & 15);
                s[j] = (half ? hi : __uint_as_float(v[j])) * sl;
            }
            if (j0 + (i + 1) * LT_KEYS > limit_lo + 1 || j0 + (i + 1) * LT_KEYS > j1) {
#pragma unroll
                for (int j = 0; j < 16; ++j)
                    if (key > sh->limit[half * 16 + j] || key >= j1) s[j] = -INFINITY;
            }
            bool over = false;
#pragma unroll
            for (int j = 0; j < 16; ++j) over |= s[j] > top[j] + LT_SLACK;
            if (softmax_any(over || !ok || *failed)) {
                if (softmax_any(!ok || *failed)) { ok = false; break; }
                float m[16];
#pragma unroll
                for (int j = 0; j < 16; ++j) m[j] = s[j];
                sh->red[quad][lane] = reduce_transposed(m, lane, [](float x, float y) { return fmaxf(x, y); });
#pragma unroll
                for (int j = 0; j < 16; ++j) m[j] = top[j];
                softmax_any(false);
                if (quad == 0) {  // lane L serves row L
                    const float best = fmaxf(fmaxf(sh->red[0][lane], sh->red[1][lane]), fmaxf(sh->red[2][lane], sh->red[3][lane]));
                    const float old = i == 0 ? -1e30f : sh->top[lane], now = fmaxf(old, best);
                    sh->top[lane] = now;
                    sh->corr[lane] = exp2f(old - now);
                }
                softmax_any(false);
#pragma unroll
                for (int j = 0; j < 16; ++j) {
                    top[j] = sh->top[half * 16 + j];
                    sum[j] *= sh->corr[half * 16 + j];
                }
                if (i > 0) {  // the sums so far, once the products that make them have finished
                    ok = bar_wait(&sh->odone[b ^ 1], ((i - 1) >> 1) & 1, failed);
                    if (softmax_any(!ok)) { ok = false; break; }
                    asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
                    for (int m2 = 0; m2 < 2 * p.mtiles; ++m2) {
                        tmem_ld32(v, tmem_o + quad_addr + (uint32_t)(m2 * LT_ROWS));
                        tmem_wait_ld(v);
#pragma unroll
                        for (int c = 0; c < 32; ++c) v[c] = __float_as_uint(__uint_as_float(v[c]) * sh->corr[c]);
                        tmem_st32(tmem_o + quad_addr + (uint32_t)(m2 * LT_ROWS), v);
                    }
                    asm volatile("tcgen05.wait::st.sync.aligned;\n" ::: "memory");
                    softmax_any(false);  // corr has been read
                }
            }
            // the weights' buffer is free when the products of the tile before last have finished
            if (i >= 2) ok = bar_wait(&sh->odone[b], ((i >> 1) - 1) & 1, failed) && ok;
            uint32_t hi[8], lo[8];
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                const float x = exp2f(s[2 * j] - top[2 * j]), y = exp2f(s[2 * j + 1] - top[2 * j + 1]);
                sum[2 * j] += x;
                sum[2 * j + 1] += y;
                const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
                const __nv_bfloat162 l = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
                hi[j] = *reinterpret_cast<const uint32_t *>(&h);
                lo[j] = *reinterpret_cast<const uint32_t *>(&l);
            }
            uint8_t *pr = pbuf + b * LT_PBUF + key_in * 128;
            const int sw = key_in & 7;
#pragma unroll
            for (int c = 0; c < 2; ++c) {
                *reinterpret_cast<uint4 *>(pr + (((half * 2 + c) ^ sw) << 4)) = make_uint4(hi[4 * c], hi[4 * c + 1], hi[4 * c + 2], hi[4 * c + 3]);
                *reinterpret_cast<uint4 *>(pr + (((4 + half * 2 + c) ^ sw) << 4)) = make_uint4(lo[4 * c], lo[4 * c + 1], lo[4 * c + 2], lo[4 * c + 3]);
            }
            asm volatile("fence.proxy.async.shared::cta;\n" ::: "memory");
            asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
            __syncwarp();
            if (lane == 0) bar_arrive(&sh->pfull[b]);
        }
        const float s_all = reduce_transposed(sum, lane, [](float x, float y) { return x + y; });
        softmax_any(false);
        sh->red[quad][lane] = s_all;
        if (tiles > 0) ok = bar_wait(&sh->odone[(tiles - 1) & 1], ((tiles - 1) >> 1) & 1, failed) && ok;
        if (!softmax_any(!ok)) {
            asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
            const size_t out0 = (size_t)rrow * rows + r0;
            const int live = min(LT_ROWS, rows - r0);
            if (quad == 0) {  // lane L serves row L
                const float l = (sh->red[0][lane] + sh->red[1][lane]) + (sh->red[2][lane] + sh->red[3][lane]);
                if (a.nsplit > 1 && lane < live) {
                    float *ml = a.part_ml + ((out0 + lane) * a.nsplit + blockIdx.x) * 2;
                    ml[0] = l > 0.f ? sh->top[lane] : -INFINITY;  // no key in sight in this run
                    ml[1] = l;
                }
                sh->corr[lane] = 1.f / l;
            }
            softmax_any(false);
            for (int m = 0; m < (tiles > 0 ? p.mtiles : 0); ++m) {
                uint32_t v[32], w[32];
                tmem_ld32(v, tmem_o + quad_addr + (uint32_t)(m * 2 * LT_ROWS));
                tmem_ld32(w, tmem_o + quad_addr + (uint32_t)(m * 2 * LT_ROWS + LT_ROWS));
                tmem_wait_ld(v);
                tmem_wait_ld(w);
                const int d = m * 128 + quad * 32 + lane;
#pragma unroll
                for (int c = 0; c < 32; ++c) {
                    const float o = __uint_as_float(v[c]) + __uint_as_float(w[c]);
                    if (c < live && d < a.rank) {
                        if (a.nsplit == 1) p.ox[(out0 + c) * a.rank + d] = __float2bfloat16_rn(o * sh->corr[c]);
                        else a.part_acc[((out0 + c) * a.nsplit + blockIdx.x) * a.rank + d] = o;
                    }
                }
            }
        }
    }

    // ---- teardown: every warp arrives here (all waits are bounded)
    asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
    __syncthreads();
    if (threadIdx.x == 0 && sh->failed) atomicExch(status, (int)AB2_ERR_TIMEOUT);
    if (warp == 1) {
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem), "r"(p.tmem_cols));
    }
}

}  // namespace

bool latent_tc_serves(int rank, int kds) { return rank <= LT_MAX_RANK && (kds + 63) / 64 <= LT_MAX_BOXES; }

int latent_tc_attention(LatentArgs &a, const __nv_bfloat16 *qx, __nv_bfloat16 *ox, int cache_rows, int nrows, int max_len, cudaStream_t s) {
    const KvLayer &l = a.kv.l;
    const int row_tiles = (a.S * a.H + LT_ROWS - 1) / LT_ROWS, units = row_tiles * nrows, sms = device_sm_count();
    a.nsplit = std::max(1, std::min(std::min(sms / units, (max_len + LT_KEYS - 1) / LT_KEYS), std::min(LATENT_PART_TILES / units, AB2_KV_MAX_SPLITS)));
    LtArgs p = {};
    p.a = a; p.ox = ox;
    p.boxes = (l.kds + 63) / 64; p.mtiles = (a.rank + 127) / 128; p.stage_boxes = std::max(p.boxes, 2 * p.mtiles);
    const size_t fixed = 1024 + (size_t)p.boxes * LT_QBOX + 2 * LT_PBUF + sizeof(LtShared), stage = (size_t)p.stage_boxes * LT_KBOX;
    p.stages = (int)std::min<size_t>(LT_MAX_STAGES, (224 * 1024 - fixed) / stage);
    AB2_REQUIRE(p.stages >= 2, AB2_ERR_UNSUPPORTED, "latent rows of %d values leave no room for two tiles", l.kds);
    p.tmem_cols = 128;
    while (p.tmem_cols < 64u + p.mtiles * 64u) p.tmem_cols <<= 1;
    int *status = nullptr;
    int rc = device_status_word(&status);
    CUtensorMap kmap, qmap;
    if (rc == AB2_OK) rc = make_x_map(&kmap, l.k, cache_rows * l.cap, l.kds, LT_KEYS);
    if (rc == AB2_OK) rc = make_x_map(&qmap, qx, nrows * a.S * a.H, l.kds, LT_ROWS);
    if (rc != AB2_OK) return rc;
    static bool configured[64] = {false};  // the attribute is per device
    int dev = 0;
    AB2_CUDA(cudaGetDevice(&dev));
    AB2_REQUIRE(dev >= 0 && dev < 64, AB2_ERR_BAD_ARG, "device index %d out of range", dev);
    if (!configured[dev]) {
        AB2_CUDA(cudaFuncSetAttribute(latent_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024));
        configured[dev] = true;
    }
    cudaError_t e = launch_kernel(latent_tc_kernel, dim3(a.nsplit, row_tiles, nrows), dim3(LT_THREADS), fixed + p.stages * stage, s, kmap, qmap, p, status);
    if (e != cudaSuccess) return fail(AB2_ERR_CUDA, "latent attention launch failed: %s", cudaGetErrorString(e));
    return AB2_OK;
}

}  // namespace ab2
