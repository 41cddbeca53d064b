// Causal attention of a prompt portion in bf16 on the 5th-generation tensor cores, over keys and values laid
// out position by position (PromptAttnArgs).  A CTA owns 128 queries of a head and walks the keys 128 at
// a time:
//
//   S[128 queries][128 keys] = Q . K^T         both K-major in shared memory
//   O[128 queries][vdim]    += (P_hi + P_lo) . V   P in tensor memory, V N-major in shared memory
//
// The softmax weights enter as two bf16 terms, the rounded weight and what rounding left, so the product carries
// them to about 16 significant bits.
//
//   warp 0       TMA producer: K and V tiles, two of each in flight
//   warp 1       MMA issue of the scores;   warp 2   MMA issue of the sums
//   warps 4-7    softmax of the even key tiles, a thread per query, with sums O_0 of their own
//   warps 8-11   softmax of the odd key tiles, with O_1; the two halves are merged at the end
// Tensor memory: S_0, S_1 (128 columns each; the weights take the place of the scores), O_0, O_1.  The
// weights are relative to a maximum per query that moves only when a score exceeds it by 2^8; then the query's
// sums are rescaled in tensor memory.
// Every wait on an mbarrier is bounded; on a time-out the CTA records AB2_ERR_TIMEOUT, stops issuing
// work, frees its tensor memory and returns.
#include <algorithm>

#include "stack.cuh"
#include "tcgen05_util.cuh"

using namespace ab2;
using namespace ab2::tc;

namespace ab2 {
int device_status_word(int **out);
namespace {

constexpr int PT_Q = 128, PT_KEYS = 128, PT_THREADS = 384, PT_BOX = 128 * 128;  // a box is 128 rows of 64 elements
constexpr int PT_SMEM = 227 * 1024;
constexpr float PT_SLACK = 8.f;  // powers of two a score may exceed the query's maximum by

struct PtShared {
    uint64_t kfull[2], kempty[2], vfull[2], vempty[2], sfull[2], pfull[2], odone[2];
    uint32_t tmem_base;
    int failed;
    float top[2][PT_Q], sum[2][PT_Q];
};

struct PtArgs {
    PromptAttnArgs a;
    int main_boxes, tail_boxes, v_boxes;
};

#define PT_REGS32(c, v) \
    c(v[0]), c(v[1]), c(v[2]), c(v[3]), c(v[4]), c(v[5]), c(v[6]), c(v[7]), c(v[8]), c(v[9]), c(v[10]), c(v[11]), c(v[12]), c(v[13]), c(v[14]), c(v[15]), \
    c(v[16]), c(v[17]), c(v[18]), c(v[19]), c(v[20]), c(v[21]), c(v[22]), c(v[23]), c(v[24]), c(v[25]), c(v[26]), c(v[27]), c(v[28]), c(v[29]), c(v[30]), c(v[31])
// 32 columns of the warp's lanes; the registers pass through the wait, so that nothing computed from them can move
// ahead of it.
__device__ __forceinline__ void tmem_ld32_start(uint32_t (&v)[32], uint32_t addr) {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x32.b32 "
        "{%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];\n"
        : PT_REGS32("=r", v) : "r"(addr));
}
__device__ __forceinline__ void tmem_ld32_wait(uint32_t (&v)[32]) { asm volatile("tcgen05.wait::ld.sync.aligned;\n" : PT_REGS32("+r", v)::"memory"); }
__device__ __forceinline__ void tmem_ld32(uint32_t (&v)[32], uint32_t addr) {
    tmem_ld32_start(v, addr);
    tmem_ld32_wait(v);
}
__device__ __forceinline__ void tmem_st32(uint32_t addr, const uint32_t (&v)[32]) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x32.b32 [%32], "
        "{%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31};\n" ::PT_REGS32("r", v), "r"(addr)
        : "memory");
}
__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}
// The first operand in tensor memory: 128 lanes, two bf16 per column.
__device__ __forceinline__ void umma_bf16_ts(uint32_t tmem_d, uint32_t tmem_a, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n .reg .pred p;\n setp.ne.b32 p, %4, 0;\n"
        " tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n}\n" ::
            "r"(tmem_d), "r"(tmem_a), "l"(bdesc), "r"(idesc), "r"(accumulate) : "memory");
}

// One tile of keys for the warp's 32 queries, a lane each: scores to weights in tensor memory.  With EDGE the keys
// past `lim` are out of sight.  o_blocks blocks of 32 columns hold sums so far.
template <bool EDGE>
__device__ __forceinline__ void softmax_tile(uint32_t s_addr, uint32_t o_addr, float sl, int lim, int o_blocks, float &top, float &sum) {
    // two buffers: the next 32 scores are on their way while these are looked at
    uint32_t v[2][32];
    float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
    tmem_ld32_start(v[0], s_addr);
#pragma unroll
    for (int c = 0; c < 4; ++c) {
        tmem_ld32_wait(v[c & 1]);
        tmem_ld32_start(v[(c + 1) & 1], s_addr + 32 * ((c + 1) & 3));  // the last one fetches the first again
#pragma unroll
        for (int k = 0; k < 32; ++k) mx[k & 3] = fmaxf(mx[k & 3], EDGE && 32 * c + k > lim ? -INFINITY : __uint_as_float(v[c & 1][k]));
    }
    tmem_ld32_wait(v[0]);
    const float best = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])) * sl;  // the scale is positive
    const float now = best > top + PT_SLACK ? best : top;
    if (__any_sync(0xffffffffu, now != top)) {
        const float corr = ex2(top - now);
        sum *= corr;
        top = now;
        // the scores came after the products of this half's last tile: its sums stand still
#pragma unroll 1
        for (int c = 0; c < o_blocks; ++c) {
            uint32_t o[32];
            tmem_ld32(o, o_addr + 32 * c);
#pragma unroll
            for (int k = 0; k < 32; ++k) o[k] = __float_as_uint(__uint_as_float(o[k]) * corr);
            tmem_st32(o_addr + 32 * c, o);
        }
    }
    float part_sum[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int c = 0; c < 4; ++c) {
        if (c > 0) tmem_ld32_wait(v[c & 1]);
        if (c < 3) tmem_ld32_start(v[(c + 1) & 1], s_addr + 32 * (c + 1));
        uint32_t w[32];
#pragma unroll
        for (int k = 0; k < 32; k += 2) {
            float x = ex2(fmaf(__uint_as_float(v[c & 1][k]), sl, -top)), y = ex2(fmaf(__uint_as_float(v[c & 1][k + 1]), sl, -top));
            if (EDGE && 32 * c + k > lim) x = 0.f;
            if (EDGE && 32 * c + k + 1 > lim) y = 0.f;
            part_sum[(k >> 1) & 3] += x + y;
            const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
            w[k >> 1] = *reinterpret_cast<const uint32_t *>(&h);
            const __nv_bfloat162 l = __floats2bfloat162_rn(x - __uint_as_float(w[k >> 1] << 16), y - __uint_as_float(w[k >> 1] & 0xffff0000u));
            w[16 + (k >> 1)] = *reinterpret_cast<const uint32_t *>(&l);
        }
        tmem_st32(s_addr + 32 * c, w);
    }
    sum += (part_sum[0] + part_sum[1]) + (part_sum[2] + part_sum[3]);
}

__global__ void __launch_bounds__(PT_THREADS, 1)
prompt_tc_kernel(const __grid_constant__ CUtensorMap kmap, const __grid_constant__ CUtensorMap tmap, const __grid_constant__ CUtensorMap vmap, PtArgs p, int *status) {
    extern __shared__ uint8_t smem_raw[];
    uint8_t *qbuf = (uint8_t *)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    const PromptAttnArgs &a = p.a;
    const int kboxes = p.main_boxes + p.tail_boxes;
    uint8_t *kbuf = qbuf + kboxes * PT_BOX, *vbuf = kbuf + 2 * kboxes * PT_BOX;
    PtShared *sh = (PtShared *)(vbuf + 2 * p.v_boxes * PT_BOX);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, head = blockIdx.y;
    const int q_lo = ((int)gridDim.x - 1 - (int)blockIdx.x) * PT_Q;  // the longest walks first
    const int tiles = (a.first + min(a.S, q_lo + PT_Q) + PT_KEYS - 1) / PT_KEYS;
    volatile int *failed = &sh->failed;

    auto load_k = [&](int j) {
        uint8_t *dst = kbuf + (j & 1) * kboxes * PT_BOX;
        bar_expect_tx(&sh->kfull[j & 1], (uint32_t)(kboxes * PT_BOX));
        for (int b = 0; b < p.main_boxes; ++b) tma_load_2d(dst + b * PT_BOX, &kmap, head * a.k_head + b * 64, j * PT_KEYS, &sh->kfull[j & 1]);
        for (int b = 0; b < p.tail_boxes; ++b) tma_load_2d(dst + (p.main_boxes + b) * PT_BOX, &tmap, b * 64, j * PT_KEYS, &sh->kfull[j & 1]);
    };
    auto load_v = [&](int j) {
        uint8_t *dst = vbuf + (j & 1) * p.v_boxes * PT_BOX;
        bar_expect_tx(&sh->vfull[j & 1], (uint32_t)(p.v_boxes * PT_BOX));
        for (int b = 0; b < p.v_boxes; ++b) tma_load_2d(dst + b * PT_BOX, &vmap, head * a.v_head + b * 64, j * PT_KEYS, &sh->vfull[j & 1]);
    };

    if (threadIdx.x == 0) {
        for (int i = 0; i < 2; ++i) {
            bar_init(&sh->kfull[i], 1); bar_init(&sh->kempty[i], 1); bar_init(&sh->vfull[i], 1); bar_init(&sh->vempty[i], 1);
            bar_init(&sh->sfull[i], 1); bar_init(&sh->pfull[i], 4); bar_init(&sh->odone[i], 1);
        }
        sh->failed = 0;
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;\n" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], 512;\n" ::"r"(sptr(&sh->tmem_base)));
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::);
    }
    pdl_wait();
    pdl_launch_dependents();
    if (threadIdx.x == 0)
        for (int j = 0; j < min(2, tiles); ++j) { load_k(j); load_v(j); }
    // the queries, in boxes like the keys; what a head or the portion does not have is zero
    for (int i = threadIdx.x; i < kboxes * PT_Q * 8; i += PT_THREADS) {
        const int ch = i & 7, r = (i >> 3) % PT_Q, b = (i >> 3) / PT_Q;
        const int d = (b < p.main_boxes ? b : b - p.main_boxes) * 64 + ch * 8;
        const bool in = q_lo + r < a.S && d < (b < p.main_boxes ? a.dim : a.tail_dims);
        const uint4 v = in ? *reinterpret_cast<const uint4 *>(a.q + (size_t)(q_lo + r) * a.q_stride + (size_t)head * (a.dim + a.tail_dims) + (b < p.main_boxes ? d : a.dim + d))
                           : make_uint4(0u, 0u, 0u, 0u);
        *reinterpret_cast<uint4 *>(qbuf + b * PT_BOX + r * 128 + ((ch ^ (r & 7)) << 4)) = v;
    }
    asm volatile("fence.proxy.async.shared::cta;\n" ::: "memory");
    asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
    const uint32_t tmem = sh->tmem_base, tmem_o = tmem + 2 * PT_KEYS;  // O_0 and O_1 128 columns apart
    constexpr uint32_t IDESC = (1u << 4) | (1u << 7) | (1u << 10) | ((128u >> 4) << 24);
    if (warp == 0) {
        // ---------------------------------------------------------- TMA producer
        if (lane == 0)
            for (int j = 2; j < tiles && !*failed; ++j) {
                if (!bar_wait(&sh->kempty[j & 1], ((j >> 1) & 1) ^ 1, failed)) break;
                load_k(j);
                if (!bar_wait(&sh->vempty[j & 1], ((j >> 1) & 1) ^ 1, failed)) break;
                load_v(j);
            }
    } else if (warp == 1) {
        // ---------------------------------------------------------- scores
        const uint32_t idesc = IDESC | ((uint32_t)(PT_KEYS >> 3) << 17);
        for (int j = 0; j < tiles; ++j) {
            if (!warp_wait(&sh->kfull[j & 1], (j >> 1) & 1, failed)) break;
            // the weights that lie in this score buffer have been multiplied
            if (j >= 2 && !warp_wait(&sh->odone[j & 1], ((j >> 1) - 1) & 1, failed)) break;
            asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
            if (elect_one()) {
                for (int b = 0; b < kboxes; ++b) {
                    const uint64_t qd = umma_desc(sptr(qbuf + b * PT_BOX)), kd = umma_desc(sptr(kbuf + ((j & 1) * kboxes + b) * PT_BOX));
#pragma unroll
                    for (int k = 0; k < 4; ++k)  // descriptors count in 16 bytes
                        umma_bf16(tmem + (uint32_t)((j & 1) * PT_KEYS), qd + (uint64_t)(2 * k), kd + (uint64_t)(2 * k), idesc, (b | k) != 0);
                }
                umma_commit(&sh->kempty[j & 1]);
                umma_commit(&sh->sfull[j & 1]);
            }
            __syncwarp();
        }
    } else if (warp == 2) {
        // ---------------------------------------------------------- sums
        const uint32_t idesc = IDESC | (1u << 16) | ((uint32_t)(p.v_boxes * 64 >> 3) << 17);
        for (int j = 0; j < tiles; ++j) {
            if (!warp_wait(&sh->vfull[j & 1], (j >> 1) & 1, failed) || !warp_wait(&sh->pfull[j & 1], (j >> 1) & 1, failed)) break;
            asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
            if (elect_one()) {
                const uint64_t vd = umma_desc_mn(sptr(vbuf + (j & 1) * p.v_boxes * PT_BOX), PT_BOX);
                const uint32_t w = tmem + (uint32_t)((j & 1) * PT_KEYS), o = tmem_o + (uint32_t)((j & 1) * 128);
#pragma unroll
                for (int k = 0; k < PT_KEYS / 16; ++k) {
                    const uint32_t at = w + (uint32_t)((k >> 1) * 32 + (k & 1) * 8);  // 32 keys: 16 columns of rounded weights, 16 of the rest
                    umma_bf16_ts(o, at, vd + (uint64_t)(k * (2048 >> 4)), idesc, j >= 2 || k > 0);
                    umma_bf16_ts(o, at + 16, vd + (uint64_t)(k * (2048 >> 4)), idesc, 1);
                }
                umma_commit(&sh->vempty[j & 1]);
                umma_commit(&sh->odone[j & 1]);
            }
            __syncwarp();
        }
    } else if (warp >= 4) {
        // ---------------------------------------------------------- softmax
        const int part = (warp - 4) >> 2, quad = warp & 3, r = quad * 32 + lane;
        const int pos = a.first + q_lo + r;
        const uint32_t quad_addr = (uint32_t)(quad * 32) << 16, s_addr = tmem + quad_addr + (uint32_t)(part * PT_KEYS), o_addr = tmem_o + quad_addr + (uint32_t)(part * 128);
        const float sl = a.scale * 1.44269504088896341f;  // scores in powers of two
        float top = -1e30f, sum = 0.f;
        bool ok = true;
        for (int j = part; j < tiles; j += 2) {
            ok = warp_wait(&sh->sfull[part], (j >> 1) & 1, failed);
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
            const bool edge = (j + 1) * PT_KEYS - 1 > a.first + q_lo;
            const int lim = pos - j * PT_KEYS;  // the last key of the tile in sight
            if (edge) softmax_tile<true>(s_addr, o_addr, sl, lim, j >= 2 ? p.v_boxes * 2 : 0, top, sum);
            else softmax_tile<false>(s_addr, o_addr, sl, lim, j >= 2 ? p.v_boxes * 2 : 0, top, sum);
            asm volatile("tcgen05.wait::st.sync.aligned;\n" ::: "memory");
            asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
            __syncwarp();
            if (lane == 0) bar_arrive(&sh->pfull[part]);
        }
        sh->top[part][r] = top;
        sh->sum[part][r] = sum;
        const int mine = (tiles - part + 1) / 2;  // tiles of this half
        if (ok && mine > 0) ok = warp_wait(&sh->odone[part], (mine - 1) & 1, failed);
        asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
        asm volatile("barrier.cta.sync 1, 256;\n" ::: "memory");
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
        if (!*failed) {
            // both halves of the warps store: value boxes of 64 dimensions in turn
            const float t0 = sh->top[0][r], t1 = sh->top[1][r], t = fmaxf(t0, t1);
            float f0 = ex2(t0 - t), f1 = tiles > 1 ? ex2(t1 - t) : 0.f;
            float scale = 1.f / (f0 * sh->sum[0][r] + f1 * sh->sum[1][r]);
            const int qi = q_lo + r;
            if (a.gate && qi < a.S) scale /= 1.f + expf(-__bfloat162float(a.gate[(size_t)qi * a.gate_stride + head]));
            f0 *= scale;
            f1 *= scale;
            __nv_bfloat16 *dst = a.out + (size_t)qi * a.out_stride + (size_t)head * a.vdim;
#pragma unroll 1
            for (int c = part; c < p.v_boxes * 2; c += 2) {
                uint32_t v[32], w[32];
                __syncwarp();
                tmem_ld32(v, tmem_o + quad_addr + 32 * c);
                if (tiles > 1) tmem_ld32(w, tmem_o + quad_addr + 128 + 32 * c);
                else
#pragma unroll
                    for (int k = 0; k < 32; ++k) w[k] = 0u;
#pragma unroll
                for (int k = 0; k < 32; k += 8) {
                    uint32_t o[4];
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const int n = k + 2 * e;
                        const __nv_bfloat162 q = __floats2bfloat162_rn(f0 * __uint_as_float(v[n]) + f1 * __uint_as_float(w[n]), f0 * __uint_as_float(v[n + 1]) + f1 * __uint_as_float(w[n + 1]));
                        o[e] = *reinterpret_cast<const uint32_t *>(&q);
                    }
                    if (qi < a.S && 32 * c + k < a.vdim) *reinterpret_cast<uint4 *>(dst + 32 * c + k) = make_uint4(o[0], o[1], o[2], o[3]);
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
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, 512;\n" ::"r"(tmem));
    }
}

size_t prompt_tc_smem(const PtArgs &p) { return 1024 + (size_t)(3 * (p.main_boxes + p.tail_boxes) + 2 * p.v_boxes) * PT_BOX + sizeof(PtShared); }

}  // namespace

bool prompt_tc_serves(const PromptAttnArgs &a) {
    const PtArgs p = {a, (a.dim + 63) / 64, (a.tail_dims + 63) / 64, (a.vdim + 63) / 64};
    return a.scale >= 0.f && a.dim % 8 == 0 && a.tail_dims % 8 == 0 && a.vdim % 8 == 0 && p.v_boxes <= 2 && prompt_tc_smem(p) <= PT_SMEM && a.q_stride % 8 == 0 &&
           a.k_stride % 8 == 0 && a.v_stride % 8 == 0 && a.tail_stride % 8 == 0 && a.k_head % 8 == 0 && a.v_head % 8 == 0 && a.out_stride % 8 == 0 &&
           (((uintptr_t)a.q | (uintptr_t)a.k | (uintptr_t)a.v | (uintptr_t)a.tail | (uintptr_t)a.out) & 15) == 0;
}

int prompt_tc_attention(const PromptAttnArgs &a, cudaStream_t s) {
    const PtArgs p = {a, (a.dim + 63) / 64, (a.tail_dims + 63) / 64, (a.vdim + 63) / 64};
    int *status = nullptr;
    int rc = device_status_word(&status);
    CUtensorMap kmap, tmap, vmap;
    const int L = a.first + a.S;
    if (rc == AB2_OK) rc = make_x_map(&kmap, a.k, L, (a.heads - 1) * a.k_head + a.dim, PT_KEYS, a.k_stride);
    if (rc == AB2_OK) rc = a.tail_dims > 0 ? make_x_map(&tmap, a.tail, L, a.tail_dims, PT_KEYS, a.tail_stride) : make_x_map(&tmap, a.k, L, a.dim, PT_KEYS, a.k_stride);
    if (rc == AB2_OK) rc = make_x_map(&vmap, a.v, L, (a.heads - 1) * a.v_head + a.vdim, PT_KEYS, a.v_stride);
    if (rc != AB2_OK) return rc;
    static bool configured[64] = {false};  // the attribute is per device
    int dev = 0;
    AB2_CUDA(cudaGetDevice(&dev));
    AB2_REQUIRE(dev >= 0 && dev < 64, AB2_ERR_BAD_ARG, "device index %d out of range", dev);
    if (!configured[dev]) {
        AB2_CUDA(cudaFuncSetAttribute(prompt_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, PT_SMEM));
        configured[dev] = true;
    }
    cudaError_t e = launch_kernel(prompt_tc_kernel, dim3((a.S + PT_Q - 1) / PT_Q, a.heads), dim3(PT_THREADS), prompt_tc_smem(p), s, kmap, tmap, vmap, p, status);
    if (e != cudaSuccess) return fail(AB2_ERR_CUDA, "prompt attention launch failed: %s", cudaGetErrorString(e));
    return AB2_OK;
}

}  // namespace ab2
