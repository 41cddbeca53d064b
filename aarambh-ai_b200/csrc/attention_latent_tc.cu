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
//   warp 0     TMA producer: tiles of 64 keys in chunks of 128 dimensions (two boxes of 64, 128-byte swizzle),
//              a ring of chunks; what the row does not have arrives as zeros.  Keys of earlier steps are
//              requested before the dependency wait.
//   warp 1     MMA issue of the scores, chunk by chunk as they arrive
//   warp 10    MMA issue of the sums, chunk by chunk (each frees its chunk)
//   warps 2-9  softmax, two per tensor-memory quadrant with 16 rows each: a lane holds one key and eight rows,
//              weights relative to a maximum per row that moves only when a score exceeds it by 2^8 (then
//              the sums in tensor memory are rescaled), and the result at the end
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

constexpr int LT_KEYS = 64, LT_ROWS = LATENT_ROWS, LT_SOFT_WARPS = 8, LT_THREADS = 96 + 32 * LT_SOFT_WARPS, LT_MAX_SLOTS = 12;
constexpr int LT_KBOX = LT_KEYS * 128, LT_SLOT = 2 * LT_KBOX, LT_QBOX = LT_ROWS * 128, LT_PBUF = LT_KEYS * 128;
constexpr int LT_MAX_BOXES = 9, LT_MAX_RANK = 512, LT_SMEM = 227 * 1024;
constexpr float LT_SLACK = 8.f;  // powers of two a score may exceed the row's maximum by

struct LtShared {
    uint64_t full[LT_MAX_SLOTS], empty[LT_MAX_SLOTS], qfull;
    uint64_t sfull[2], sfree[2], pfull, odone;
    uint32_t tmem_base;
    int failed;
    int limit[LT_ROWS];       // last position a row sees
    float red[4][LT_ROWS], top[LT_ROWS], corr[LT_ROWS];
};

struct LtArgs {
    LatentArgs a;
    __nv_bfloat16 *ox;
    int boxes, chunks, mtiles, slots;  // of a cache row: boxes of 64 and chunks of 128 dimensions; chunks that are latent
    uint32_t tmem_cols;
};

// A position in the ring of chunks.
struct LtSlot {
    int slot = 0;
    uint32_t phase = 0;
    __device__ __forceinline__ void next(int slots) {
        if (++slot == slots) { slot = 0; phase ^= 1; }
    }
};

constexpr uint32_t LT_IDESC = (1u << 4) | (1u << 7) | (1u << 10);  // f32 sums of bf16 products
// Barrier of the softmax warps; returns whether any of them passed true.
__device__ __forceinline__ bool softmax_any(bool p) {
    uint32_t r;
    asm volatile("{\n .reg .pred p, q;\n setp.ne.b32 p, %1, 0;\n barrier.cta.red.or.pred q, 1, 256, p;\n selp.u32 %0, 1, 0, q;\n}\n" : "=r"(r) : "r"((uint32_t)p) : "memory");
    return r != 0;
}
#define LT_REGS16(c, v) \
    c(v[0]), c(v[1]), c(v[2]), c(v[3]), c(v[4]), c(v[5]), c(v[6]), c(v[7]), c(v[8]), c(v[9]), c(v[10]), c(v[11]), c(v[12]), c(v[13]), c(v[14]), c(v[15])
// Loads of 16 or 8 columns of the warp's lanes.  The registers pass through the wait, so that nothing computed from
// them can move ahead of it.
__device__ __forceinline__ void tmem_ld16(uint32_t (&v)[16], uint32_t addr) {
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];\n" : LT_REGS16("=r", v) : "r"(addr));
    asm volatile("tcgen05.wait::ld.sync.aligned;\n" : LT_REGS16("+r", v)::"memory");
}
__device__ __forceinline__ void tmem_st16(uint32_t addr, const uint32_t (&v)[16]) {
    asm volatile("tcgen05.st.sync.aligned.32x32b.x16.b32 [%16], {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15};\n" ::LT_REGS16("r", v), "r"(addr) : "memory");
}
__device__ __forceinline__ void tmem_ld8_pair(uint32_t (&v)[8], uint32_t (&w)[8], uint32_t va, uint32_t wa) {
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x8.b32 {%0,%1,%2,%3,%4,%5,%6,%7}, [%8];\n"
                 : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]) : "r"(va));
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x8.b32 {%0,%1,%2,%3,%4,%5,%6,%7}, [%8];\n"
                 : "=r"(w[0]), "=r"(w[1]), "=r"(w[2]), "=r"(w[3]), "=r"(w[4]), "=r"(w[5]), "=r"(w[6]), "=r"(w[7]) : "r"(wa));
    asm volatile("tcgen05.wait::ld.sync.aligned;\n"
                 : "+r"(v[0]), "+r"(v[1]), "+r"(v[2]), "+r"(v[3]), "+r"(v[4]), "+r"(v[5]), "+r"(v[6]), "+r"(v[7]), "+r"(w[0]), "+r"(w[1]), "+r"(w[2]),
                   "+r"(w[3]), "+r"(w[4]), "+r"(w[5]), "+r"(w[6]), "+r"(w[7])::"memory");
}
__device__ __forceinline__ void put(float *p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16 *p, float v) { *p = __float2bfloat16_rn(v); }
// Rows [c, c_end) of the sums in tensor memory (times scale[row]) to dst[row * step + dimension]; this lane has
// the dimensions d, d + 128, ...
template <typename T>
__device__ __forceinline__ void store_rows(T *dst, size_t step, uint32_t o, int c, int c_end, int d, int rank, int mtiles, const float *scale) {
    dst += c * step + d;
#pragma unroll 1
    for (; c < c_end; c += 8, dst += 8 * step) {
#pragma unroll 1
        for (int m = 0; m < mtiles; ++m) {
            uint32_t v[8], w[8];
            __syncwarp();
            tmem_ld8_pair(v, w, o + (uint32_t)(m * 2 * LT_ROWS + c), o + (uint32_t)(m * 2 * LT_ROWS + LT_ROWS + c));
            if (m * 128 + d >= rank) continue;
            T *q = dst + m * 128;
#pragma unroll
            for (int k = 0; k < 8; ++k, q += step)
                if (c + k < c_end) put(q, (__uint_as_float(v[k]) + __uint_as_float(w[k])) * (scale ? scale[c + k] : 1.f));
        }
    }
}

// Reduces eight values per lane over the half warp's 16 lanes: lane L ends with the result of its value
// (L & 15) >> 1.
template <class Op>
__device__ __forceinline__ float reduce_transposed(const float (&in)[8], int lane, Op op) {
    float v[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = in[j];
#pragma unroll
    for (int w = 4; w > 0; w >>= 1) {
        const bool up = lane & (2 * w);
#pragma unroll
        for (int j = 0; j < w; ++j) {
            const float send = up ? v[j] : v[j + w], keep = up ? v[j + w] : v[j];
            v[j] = op(keep, __shfl_xor_sync(0xffffffffu, send, 2 * w));
        }
    }
    return op(v[0], __shfl_xor_sync(0xffffffffu, v[0], 1));
}

__global__ void __launch_bounds__(LT_THREADS, 1)
latent_tc_kernel(const __grid_constant__ CUtensorMap kmap, const __grid_constant__ CUtensorMap qmap, LtArgs p, int *status) {
    extern __shared__ uint8_t smem_raw[];
    uint8_t *ring = (uint8_t *)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    const LatentArgs &a = p.a;
    uint8_t *qbuf = ring + p.slots * LT_SLOT, *pbuf = qbuf + p.boxes * LT_QBOX;
    LtShared *sh = (LtShared *)(pbuf + LT_PBUF);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    volatile int *failed = &sh->failed;

    const int rrow = blockIdx.z, row = kv_row(a.kv, a.row0, rrow), len = a.kv.lens[row];  // committed by earlier steps
    const int rows = a.S * a.H, r0 = blockIdx.y * LT_ROWS;
    const int n = len + min(rows - 1, r0 + LT_ROWS - 1) / a.H + 1;
    const int per = ((n + a.nsplit - 1) / a.nsplit + LT_KEYS - 1) / LT_KEYS * LT_KEYS;
    const int j0 = (int)blockIdx.x * per, j1 = min(n, j0 + per), tiles = j1 > j0 ? (j1 - j0 + LT_KEYS - 1) / LT_KEYS : 0;

    if (threadIdx.x == 0) {
        for (int i = 0; i < p.slots; ++i) { bar_init(&sh->full[i], 1); bar_init(&sh->empty[i], 1); }
        bar_init(&sh->qfull, 1);
        bar_init(&sh->sfull[0], 1); bar_init(&sh->sfull[1], 1);
        bar_init(&sh->sfree[0], LT_SOFT_WARPS); bar_init(&sh->sfree[1], LT_SOFT_WARPS);
        bar_init(&sh->pfull, LT_SOFT_WARPS);
        bar_init(&sh->odone, 1);
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
            LtSlot put;
            for (int i = 0; i < tiles * p.chunks && !*failed; ++i) {
                const int chunk = i % p.chunks, key = j0 + i / p.chunks * LT_KEYS, nb = min(2, p.boxes - 2 * chunk);
                if (!waited && (i >= p.slots || key + LT_KEYS > len)) start();  // the tile has keys of this step
                if (!bar_wait(&sh->empty[put.slot], put.phase ^ 1, failed)) break;
                uint8_t *dst = ring + put.slot * LT_SLOT;
                bar_expect_tx(&sh->full[put.slot], (uint32_t)(nb * LT_KBOX));
                for (int b = 0; b < nb; ++b) tma_load_2d(dst + b * LT_KBOX, &kmap, (2 * chunk + b) * 64, row * a.kv.l.cap + key, &sh->full[put.slot]);
                put.next(p.slots);
            }
            if (!waited) start();
        }
    } else if (warp == 1) {
        // ---------------------------------------------------------- scores
        constexpr uint32_t IDESC = LT_IDESC | ((uint32_t)(LT_ROWS >> 3) << 17) | ((64u >> 4) << 24);
        LtSlot at;
        bool ok = tiles > 0 && warp_wait(&sh->qfull, 0, failed);
        for (int i = 0; ok && i < tiles; ++i) {
            ok = warp_wait(&sh->sfree[i & 1], ((i >> 1) & 1) ^ 1, failed);  // the buffer's last scores have been read
            const uint32_t d = tmem + (uint32_t)((i & 1) * LT_ROWS);
            for (int c = 0; ok && c < p.chunks; ++c) {
                ok = warp_wait(&sh->full[at.slot], at.phase, failed);
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
                if (elect_one()) {
                    const uint64_t a0 = umma_desc(sptr(ring + at.slot * LT_SLOT)), b0 = umma_desc(sptr(qbuf + 2 * c * LT_QBOX));
                    const bool two = 2 * c + 1 < p.boxes;
#pragma unroll
                    for (int k = 0; k < 8; ++k)  // descriptors count in 16 bytes
                        if (k < 4 || two)
                            umma_bf16(d, a0 + (uint64_t)((k >> 2) * (LT_KBOX >> 4) + 2 * (k & 3)), b0 + (uint64_t)((k >> 2) * (LT_QBOX >> 4) + 2 * (k & 3)), IDESC, k > 0 || c > 0);
                    if (c >= p.mtiles) umma_commit(&sh->empty[at.slot]);  // no latents in it
                    if (c + 1 == p.chunks) umma_commit(&sh->sfull[i & 1]);
                }
                __syncwarp();
                at.next(p.slots);
            }
        }
    } else if (warp == 2 + LT_SOFT_WARPS) {
        // ---------------------------------------------------------- sums
        constexpr uint32_t IDESC = LT_IDESC | (1u << 15) | (1u << 16) | ((uint32_t)((2 * LT_ROWS) >> 3) << 17) | ((128u >> 4) << 24);
        LtSlot at;
        for (int i = 0; i < tiles; ++i) {
            if (!warp_wait(&sh->pfull, i & 1, failed)) break;
            asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
            for (int m = 0; m < p.chunks; ++m, at.next(p.slots)) {
                if (m >= p.mtiles) continue;
                if (elect_one()) {
                    const uint64_t a0 = umma_desc_mn(sptr(ring + at.slot * LT_SLOT), LT_KBOX), b0 = umma_desc_mn(sptr(pbuf), LT_PBUF);
#pragma unroll
                    for (int k = 0; k < LT_KEYS / 16; ++k)
                        umma_bf16(tmem_o + (uint32_t)(m * 2 * LT_ROWS), a0 + (uint64_t)(k * (2048 >> 4)), b0 + (uint64_t)(k * (2048 >> 4)), IDESC, k > 0 || i > 0);
                    umma_commit(&sh->empty[at.slot]);
                    if (m + 1 == p.mtiles) umma_commit(&sh->odone);
                }
                __syncwarp();
            }
        }
    } else {
        // ---------------------------------------------------------- softmax
        const int quad = warp & 3, half = lane >> 4, key_in = quad * 16 + (lane & 15);
        const int part = (warp - 2) >> 2, row_at = part * 16 + half * 8;      // the first of this lane's eight rows
        const int my_row = row_at + ((lane & 15) >> 1);                        // the row whose reduction it ends with
        const uint32_t quad_addr = (uint32_t)(quad * 32) << 16;
        const float sl = a.scale * 1.44269504088896341f;  // scores in powers of two
        const int live = min(LT_ROWS, rows - r0);
        float top[8], sum[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) { top[j] = -1e30f; sum[j] = 0.f; }
        const int limit_lo = sh->limit[0];  // limits grow with the row
        auto larger = [](float x, float y) { return fmaxf(x, y); };
        auto add = [](float x, float y) { return x + y; };
        pdl_wait();
        bool ok = true;
        for (int i = 0; i < tiles; ++i) {
            const int key = j0 + i * LT_KEYS + key_in;
            ok = bar_wait(&sh->sfull[i & 1], (i >> 1) & 1, failed);
            asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
            __syncwarp();
            uint32_t v[16];
            tmem_ld16(v, tmem + quad_addr + (uint32_t)((i & 1) * LT_ROWS + part * 16));
            asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
            __syncwarp();
            if (lane == 0) bar_arrive(&sh->sfree[i & 1]);
            float s[8];
#pragma unroll
            for (int j = 0; j < 8; ++j) {  // the upper half warp takes the upper eight rows of the lower half's keys
                const float hi = __shfl_sync(0xffffffffu, __uint_as_float(v[8 + j]), lane & 15);
                s[j] = (half ? hi : __uint_as_float(v[j])) * sl;
            }
            if (j0 + (i + 1) * LT_KEYS > limit_lo + 1 || j0 + (i + 1) * LT_KEYS > j1) {
#pragma unroll
                for (int j = 0; j < 8; ++j)
                    if (key > sh->limit[row_at + j] || key >= j1) s[j] = -INFINITY;
            }
            bool over = false;
#pragma unroll
            for (int j = 0; j < 8; ++j) over |= s[j] > top[j] + LT_SLACK;
            if (softmax_any(over || !ok || *failed)) {
                if (softmax_any(!ok || *failed)) { ok = false; break; }
                const float best = reduce_transposed(s, lane, larger);
                if ((lane & 1) == 0) sh->red[quad][my_row] = best;
                softmax_any(false);
                if (warp == 2) {  // lane L serves row L
                    const float all = fmaxf(fmaxf(sh->red[0][lane], sh->red[1][lane]), fmaxf(sh->red[2][lane], sh->red[3][lane]));
                    const float old = i == 0 ? -1e30f : sh->top[lane], now = fmaxf(old, all);
                    sh->top[lane] = now;
                    sh->corr[lane] = exp2f(old - now);
                }
                softmax_any(false);
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    top[j] = sh->top[row_at + j];
                    sum[j] *= sh->corr[row_at + j];
                }
                if (i > 0) {  // the sums so far, once the products that make them have finished
                    ok = bar_wait(&sh->odone, (i - 1) & 1, failed);
                    if (softmax_any(!ok)) { ok = false; break; }
                    asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
#pragma unroll 1
                    for (int m = 0; m < 2 * p.mtiles; ++m) {  // this warp's 16 rows, of the rounded weights and of the rest
                        const uint32_t at = tmem_o + quad_addr + (uint32_t)(m * LT_ROWS + part * 16);
                        tmem_ld16(v, at);
#pragma unroll
                        for (int c = 0; c < 16; ++c) v[c] = __float_as_uint(__uint_as_float(v[c]) * sh->corr[part * 16 + c]);
                        tmem_st16(at, v);
                    }
                    asm volatile("tcgen05.wait::st.sync.aligned;\n" ::: "memory");
                    softmax_any(false);  // corr has been read
                }
            }
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float x = exp2f(s[2 * j] - top[2 * j]), y = exp2f(s[2 * j + 1] - top[2 * j + 1]);
                sum[2 * j] += x;
                sum[2 * j + 1] += y;
                const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
                const __nv_bfloat162 l = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
                hi[j] = *reinterpret_cast<const uint32_t *>(&h);
                lo[j] = *reinterpret_cast<const uint32_t *>(&l);
            }
            // the weights' buffer is free when the products of the tile before have finished
            if (i > 0) ok = bar_wait(&sh->odone, (i - 1) & 1, failed) && ok;
            uint8_t *pr = pbuf + key_in * 128;
            const int sw = key_in & 7, chunk = part * 2 + half;
            *reinterpret_cast<uint4 *>(pr + ((chunk ^ sw) << 4)) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
            *reinterpret_cast<uint4 *>(pr + (((4 + chunk) ^ sw) << 4)) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
            asm volatile("fence.proxy.async.shared::cta;\n" ::: "memory");
            asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
            __syncwarp();
            if (lane == 0) bar_arrive(&sh->pfull);
        }
        const float s_all = reduce_transposed(sum, lane, add);
        softmax_any(false);
        if ((lane & 1) == 0) sh->red[quad][my_row] = s_all;
        if (tiles > 0) ok = bar_wait(&sh->odone, (tiles - 1) & 1, failed) && ok;
        if (!softmax_any(!ok)) {
            asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
            const size_t out0 = (size_t)rrow * rows + r0;
            if (warp == 2) {  // lane L serves row L
                const float l = (sh->red[0][lane] + sh->red[1][lane]) + (sh->red[2][lane] + sh->red[3][lane]);
                if (a.nsplit > 1 && lane < live) {
                    float *ml = a.part_ml + ((out0 + lane) * a.nsplit + blockIdx.x) * 2;
                    ml[0] = l > 0.f ? sh->top[lane] : -INFINITY;  // no key in sight in this run
                    ml[1] = l;
                }
                sh->corr[lane] = 1.f / l;
            }
            softmax_any(false);
            // this warp's 16 rows, eight at a time; the code is short because a launch runs it once
            const int c_end = min(live, part * 16 + 16);
            if (a.nsplit == 1) store_rows(p.ox + out0 * a.rank, (size_t)a.rank, tmem_o + quad_addr, part * 16, c_end, quad * 32 + lane, a.rank, tiles > 0 ? p.mtiles : 0, sh->corr);
            else store_rows(a.part_acc + (out0 * a.nsplit + blockIdx.x) * a.rank, (size_t)a.nsplit * a.rank, tmem_o + quad_addr, part * 16, c_end, quad * 32 + lane, a.rank, tiles > 0 ? p.mtiles : 0, nullptr);
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
    p.boxes = (l.kds + 63) / 64; p.chunks = (p.boxes + 1) / 2; p.mtiles = (a.rank + 127) / 128;
    const size_t fixed = 1024 + (size_t)p.boxes * LT_QBOX + LT_PBUF + sizeof(LtShared);
    p.slots = (int)std::min<size_t>(LT_MAX_SLOTS, (LT_SMEM - fixed) / LT_SLOT);
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
        AB2_CUDA(cudaFuncSetAttribute(latent_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, LT_SMEM));
        configured[dev] = true;
    }
    cudaError_t e = launch_kernel(latent_tc_kernel, dim3(a.nsplit, row_tiles, nrows), dim3(LT_THREADS), fixed + (size_t)p.slots * LT_SLOT, s, kmap, qmap, p, status);
    if (e != cudaSuccess) return fail(AB2_ERR_CUDA, "latent attention launch failed: %s", cudaGetErrorString(e));
    return AB2_OK;
}

}  // namespace ab2
