// Grouped-query attention over a sliding window: query i sees the keys j with 0 <= i - j < window.
// Keys and values are in f32 or bf16, key and value sizes may differ, and a (sequence, head) keeps
// only the slots a window needs: position p lives in slot p mod cap.
//
//   window_prep_kernel         rotation of the leading dimensions in adjacent pairs, division by the
//                              root mean square, value mixing, store into the ring
//   window_attn_kernel         f32 arithmetic on CUDA cores: decode (the window split over CTAs,
//                              log-sum-exp merge), f32 models, unusual head sizes
//   window_attn_mma_kernel     prompts in bf16 on the warp-level tensor cores; also over explicit keys (prompt_attention)
//   window_decode_mma_kernel   decode in bf16, preparation included, on the warp-level tensor cores
//
// Scores, softmax weights and sums are f32 throughout.  The tensor-core kernel multiplies the
// weights with the values as two bf16 terms (the rounded weight and what rounding left), so the
// product carries them to about 16 significant bits instead of 8.
#include <algorithm>
#include <cfloat>
#include <type_traits>

#include "stack.cuh"

using namespace ab2;

namespace ab2 {
int device_sm_count();
namespace {

constexpr int MAX_DIM = 256;

// Rotation and normalisation of one head by one warp: lane j holds the pairs j, j + 32, ... of `src`
// (NP of them at most) in u and w.
template <typename T, int NP>
__device__ __forceinline__ void rotate_normalise(const WindowPrepArgs &a, const T *src, int pos, int lane, float (&u)[NP], float (&w)[NP]) {
    const int half = (a.dim + 1) >> 1;
    float sum = 0.f;
#pragma unroll
    for (int j = 0; j < NP; ++j) {
        const int i = lane + 32 * j;
        u[j] = w[j] = 0.f;
        if (i >= half) continue;
        float x0 = to_f32(src[2 * i]), x1 = 2 * i + 1 < a.dim ? to_f32(src[2 * i + 1]) : 0.f;
        if (2 * i < a.rot_dims) {
            const size_t t = (size_t)pos * (a.rot_dims >> 1) + i;
            const float c = a.cos_t[t], sn = a.sin_t[t], r0 = x0 * c - x1 * sn, r1 = x1 * c + x0 * sn;
            x0 = r0; x1 = r1;
        }
        u[j] = x0; w[j] = x1;
        sum = fmaf(x0, x0, fmaf(x1, x1, sum));
    }
    if (!a.qk_norm) return;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    const float inv = 1.f / sqrtf(sum / (float)a.dim + a.eps);
#pragma unroll
    for (int j = 0; j < NP; ++j) { u[j] *= inv; w[j] *= inv; }
}

// One warp per (token, head): H query heads, then G key heads, then G value heads.
template <typename T>
__global__ void __launch_bounds__(256) window_prep_kernel(WindowPrepArgs a) {
    pdl_wait();
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31, vec = blockIdx.x * 8 + (threadIdx.x >> 5);
    const int s = blockIdx.y, rrow = blockIdx.z, row = kv_row(a.kv, a.row0, rrow);
    if (vec >= a.H + 2 * a.G) return;
    const KvLayer &l = a.kv.l;
    const int pos = a.kv.lens[row] + s, slot = pos % l.cap;
    const size_t tok = (size_t)rrow * a.S + s;
    T *src = (T *)a.qkv + tok * a.stride;
    if (vec >= a.H + a.G) {
        const int g = vec - a.H - a.G;
        src += (size_t)(a.H + a.G) * a.dim + (size_t)g * a.vdim;
        T *first = (T *)a.v_first + (tok * a.G + g) * a.vdim;
        T *dst = (T *)l.v + (((size_t)row * a.G + g) * l.cap + slot) * l.vds;
        for (int d = lane; d < a.vdim; d += 32) {
            float v = to_f32(src[d]);
            if (a.v_mode == 1) first[d] = src[d];
            if (a.v_mode == 2) v = (1.f - a.lambda) * v + a.lambda * to_f32(first[d]);
            dst[d] = from_f32<T>(v);
        }
        return;
    }
    src += (size_t)vec * a.dim;
    const int half = (a.dim + 1) >> 1;
    float u[MAX_DIM / 64], w[MAX_DIM / 64];
    rotate_normalise<T, MAX_DIM / 64>(a, src, pos, lane, u, w);
    T *dst = vec < a.H ? src : (T *)l.k + (((size_t)row * a.G + (vec - a.H)) * l.cap + slot) * l.kds;
#pragma unroll
    for (int j = 0; j < MAX_DIM / 64; ++j) {
        const int i = lane + 32 * j;
        if (i >= half) continue;
        dst[2 * i] = from_f32<T>(u[j]);
        if (2 * i + 1 < a.dim) dst[2 * i + 1] = from_f32<T>(w[j]);
    }
}

template <typename T> __device__ __forceinline__ void load8(const T *p, float (&f)[8]);
template <> __device__ __forceinline__ void load8<float>(const float *p, float (&f)[8]) {
    const float4 a = reinterpret_cast<const float4 *>(p)[0], b = reinterpret_cast<const float4 *>(p)[1];
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
template <> __device__ __forceinline__ void load8<__nv_bfloat16>(const __nv_bfloat16 *p, float (&f)[8]) {
    const uint4 v = *reinterpret_cast<const uint4 *>(p);
    const uint32_t r[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) { f[2 * i] = __uint_as_float(r[i] << 16); f[2 * i + 1] = __uint_as_float(r[i] & 0xffff0000u); }
}

// grid (nsplit, G * head groups, nrows * S), 128 threads.  REP query heads of one KV head per CTA;
// VPL value dimensions per lane.  The visible keys of the query are cut into nsplit runs; a warp
// takes 32 keys at a time, a lane one key in the score phase.
template <typename T, int REP, int VPL>
__global__ void __launch_bounds__(128) window_attn_kernel(WindowAttnArgs a) {
    extern __shared__ __align__(16) float dyn[];
    __shared__ float ps[4][REP][32];
    __shared__ float wm[4][REP], wl[4][REP];
    pdl_wait();
    pdl_launch_dependents();
    const KvLayer &l = a.kv.l;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float *qs = dyn, *wacc = dyn + REP * l.kds;  // [REP][kds], [4][REP][vdim]
    const int groups = (a.rep + REP - 1) / REP, kvh = blockIdx.y / groups, hg = blockIdx.y % groups;
    const int head0 = kvh * a.rep + hg * REP, nh = min(REP, a.rep - hg * REP);
    const int rrow = blockIdx.z / a.S, qi = blockIdx.z % a.S, row = kv_row(a.kv, a.row0, rrow);
    const int pos = a.kv.lens[row] + qi, lo = max(0, pos - l.window + 1), n = pos + 1 - lo;
    const int per = ((n + a.nsplit - 1) / a.nsplit + 31) & ~31;
    const int j0 = lo + (int)blockIdx.x * per, j1 = min(pos + 1, j0 + per);

    const T *q = (const T *)a.q + (size_t)blockIdx.z * a.q_stride + (size_t)head0 * a.dim;
    for (int i = threadIdx.x; i < REP * l.kds; i += 128) {
        const int hh = i / l.kds, d = i % l.kds;
        qs[i] = hh < nh && d < a.dim ? to_f32(q[(size_t)hh * a.dim + d]) : 0.f;
    }
    __syncthreads();
    const T *kb = (const T *)l.k + ((size_t)row * l.kvh + kvh) * l.cap * l.kds;
    const T *vb = (const T *)l.v + ((size_t)row * l.kvh + kvh) * l.cap * l.vds;
    float m_run[REP], l_run[REP], acc[REP][VPL];
#pragma unroll
    for (int hh = 0; hh < REP; ++hh) {
        m_run[hh] = -INFINITY;
        l_run[hh] = 0.f;
#pragma unroll
        for (int j = 0; j < VPL; ++j) acc[hh][j] = 0.f;
    }
    for (int base = j0 + warp * 32; base < j1; base += 128) {
        const int key = base + lane;
        const bool valid = key < j1;
        const T *kr = kb + (size_t)((valid ? key : j1 - 1) % l.cap) * l.kds;
        float sc[REP];
#pragma unroll
        for (int hh = 0; hh < REP; ++hh) sc[hh] = 0.f;
#pragma unroll 4
        for (int d0 = 0; d0 < l.kds; d0 += 8) {
            float kf[8];
            load8<T>(kr + d0, kf);
#pragma unroll
            for (int hh = 0; hh < REP; ++hh)
#pragma unroll
                for (int i = 0; i < 8; i += 4) {
                    const float4 qv = *reinterpret_cast<const float4 *>(&qs[hh * l.kds + d0 + i]);
                    sc[hh] = fmaf(qv.x, kf[i], sc[hh]);
                    sc[hh] = fmaf(qv.y, kf[i + 1], sc[hh]);
                    sc[hh] = fmaf(qv.z, kf[i + 2], sc[hh]);
                    sc[hh] = fmaf(qv.w, kf[i + 3], sc[hh]);
                }
        }
#pragma unroll
        for (int hh = 0; hh < REP; ++hh) {
            const float s = valid ? sc[hh] * a.scale : -INFINITY;
            float cm = s;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) cm = fmaxf(cm, __shfl_xor_sync(0xffffffffu, cm, o));
            const float m_new = fmaxf(m_run[hh], cm), corr = expf(m_run[hh] - m_new), p = valid ? expf(s - m_new) : 0.f;
            float psum = p;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) psum += __shfl_xor_sync(0xffffffffu, psum, o);
            l_run[hh] = l_run[hh] * corr + psum;
            m_run[hh] = m_new;
#pragma unroll
            for (int j = 0; j < VPL; ++j) acc[hh][j] *= corr;
            ps[warp][hh][lane] = p;
        }
        __syncwarp();
        const int nt = min(32, j1 - base);
        int slot = base % l.cap;
#pragma unroll 4
        for (int t = 0; t < nt; ++t) {
            const T *vr = vb + (size_t)slot * l.vds;
            if (++slot == l.cap) slot = 0;
            float vf[VPL];
#pragma unroll
            for (int j = 0; j < VPL; ++j) vf[j] = lane + 32 * j < a.vdim ? to_f32(vr[lane + 32 * j]) : 0.f;
#pragma unroll
            for (int hh = 0; hh < REP; ++hh) {
                const float p = ps[warp][hh][t];
#pragma unroll
                for (int j = 0; j < VPL; ++j) acc[hh][j] = fmaf(p, vf[j], acc[hh][j]);
            }
        }
        __syncwarp();
    }
#pragma unroll
    for (int hh = 0; hh < REP; ++hh) {
        if (lane == 0) { wm[warp][hh] = m_run[hh]; wl[warp][hh] = l_run[hh]; }
#pragma unroll
        for (int j = 0; j < VPL; ++j)
            if (lane + 32 * j < a.vdim) wacc[((size_t)warp * REP + hh) * a.vdim + lane + 32 * j] = acc[hh][j];
    }
    __syncthreads();
    for (int i = threadIdx.x; i < nh * a.vdim; i += 128) {
        const int hh = i / a.vdim, d = i % a.vdim;
        const float M = fmaxf(fmaxf(wm[0][hh], wm[1][hh]), fmaxf(wm[2][hh], wm[3][hh]));
        float L = 0.f, A = 0.f;
#pragma unroll
        for (int w = 0; w < 4; ++w) {
            const float e = wm[w][hh] == -INFINITY ? 0.f : expf(wm[w][hh] - M);
            L += e * wl[w][hh];
            A += e * wacc[((size_t)w * REP + hh) * a.vdim + d];
        }
        const int head = head0 + hh;
        if (a.nsplit == 1) {
            ((T *)a.out)[((size_t)blockIdx.z * a.H + head) * a.vdim + d] = from_f32<T>(A / L);
        } else {
            const size_t pi = ((size_t)rrow * a.H + head) * a.nsplit + blockIdx.x;
            a.part_acc[pi * a.vdim + d] = A;
            if (d == 0) { a.part_ml[pi * 2] = M; a.part_ml[pi * 2 + 1] = L; }
        }
    }
}

// Merge of the splits of a decode query: grid (H, nrows).
template <typename T>
__global__ void window_merge_kernel(WindowAttnArgs a) {
    pdl_wait();
    pdl_launch_dependents();
    const int head = blockIdx.x, rrow = blockIdx.y;
    const size_t p0 = ((size_t)rrow * a.H + head) * a.nsplit;
    float M = -INFINITY, L = 0.f;
    for (int i = 0; i < a.nsplit; ++i) M = fmaxf(M, a.part_ml[(p0 + i) * 2]);
    for (int i = 0; i < a.nsplit; ++i) {
        const float m = a.part_ml[(p0 + i) * 2];
        if (m != -INFINITY) L += expf(m - M) * a.part_ml[(p0 + i) * 2 + 1];
    }
    for (int d = threadIdx.x; d < a.vdim; d += blockDim.x) {
        float A = 0.f;
        for (int i = 0; i < a.nsplit; ++i) {
            const float m = a.part_ml[(p0 + i) * 2];
            if (m != -INFINITY) A += expf(m - M) * a.part_acc[(p0 + i) * a.vdim + d];
        }
        ((T *)a.out)[((size_t)rrow * a.H + head) * a.vdim + d] = from_f32<T>(A / L);
    }
}

// ---------------------------------------------------------------------------
// Prompts in bf16.  A CTA owns 64 consecutive queries of one head (16 per warp) and walks the keys
// its window reaches 64 at a time; K and V tiles are double-buffered in shared memory by cp.async
// (16-byte chunks stored at chunk ^ (row & 7)), shared by the four warps.  Head sizes are padded to
// DP / VP with zeros on the way in.
// ---------------------------------------------------------------------------
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// Two floats as bf16 pairs: the rounded values and the rounded remainders.
__device__ __forceinline__ void split_pair(float x, float y, uint32_t &hi, uint32_t &lo) {
    const __nv_bfloat16 xh = __float2bfloat16_rn(x), yh = __float2bfloat16_rn(y);
    const __nv_bfloat16 xl = __float2bfloat16_rn(x - __bfloat162float(xh)), yl = __float2bfloat16_rn(y - __bfloat162float(yh));
    hi = (uint32_t)__bfloat16_as_ushort(xh) | ((uint32_t)__bfloat16_as_ushort(yh) << 16);
    lo = (uint32_t)__bfloat16_as_ushort(xl) | ((uint32_t)__bfloat16_as_ushort(yl) << 16);
}

// The keys come from a stack cache (WindowAttnArgs: grid z is the row) or lie position by position with
// the last `tail_dims` dimensions in a matrix of their own (PromptAttnArgs).
template <int DP, int VP, class Args>
__global__ void __launch_bounds__(128) window_attn_mma_kernel(Args a) {
    extern __shared__ __align__(1024) uint8_t smem[];
    constexpr int KT = 64, KB = KT * DP * 2, VB = KT * VP * 2;
    constexpr bool EXPLICIT = std::is_same<Args, PromptAttnArgs>::value;
    pdl_wait();
    pdl_launch_dependents();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, c = lane & 3;
    const int head = blockIdx.y, rrow = blockIdx.z;
    const int q_lo = ((int)gridDim.x - 1 - (int)blockIdx.x) * 64;  // the longest key walks first
    const __nv_bfloat16 *kb, *vb, *tail = nullptr, *q0;
    size_t kst, vst, tst = 0, out_stride;
    int len, window, cap, dim, kdims, vdims, kmain;  // key dimensions from kmain on are in `tail`
    if constexpr (EXPLICIT) {
        kb = a.k + (size_t)head * a.k_head; vb = a.v + (size_t)head * a.v_head; tail = a.tail;
        kst = a.k_stride; vst = a.v_stride; tst = a.tail_stride;
        len = a.first; window = 1 << 30; cap = 1 << 30;
        dim = kdims = a.dim + a.tail_dims; kmain = a.dim; vdims = a.vdim;
        q0 = a.q + (size_t)head * dim; out_stride = a.out_stride;
    } else {
        const KvLayer &l = a.kv.l;
        const int kvh = head / a.rep, row = kv_row(a.kv, a.row0, rrow);
        kb = (const __nv_bfloat16 *)l.k + ((size_t)row * l.kvh + kvh) * l.cap * l.kds;
        vb = (const __nv_bfloat16 *)l.v + ((size_t)row * l.kvh + kvh) * l.cap * l.vds;
        kst = l.kds; vst = l.vds;
        len = a.kv.lens[row]; window = l.window; cap = l.cap;
        dim = a.dim; kdims = kmain = l.kds; vdims = l.vds;
        q0 = (const __nv_bfloat16 *)a.q + (size_t)rrow * a.S * a.q_stride + (size_t)head * dim; out_stride = (size_t)a.H * a.vdim;
    }
    const int key_lo = max(0, len + q_lo - window + 1), key_hi = len + min(a.S, q_lo + 64) - 1;

    auto load_tile = [&](int base, int buf) {
        const uint32_t ks = (uint32_t)__cvta_generic_to_shared(smem) + buf * (KB + VB), vs = ks + KB;
        const int slot0 = EXPLICIT ? base : base % cap;
        for (int i = threadIdx.x; i < KT * (DP / 8); i += 128) {
            const int r = i / (DP / 8), ch = i % (DP / 8);
            int slot = slot0 + min(r, key_hi - base);  // rows past the last key repeat it (masked below)
            if (!EXPLICIT && slot >= cap) slot -= cap;
            const __nv_bfloat16 *src = EXPLICIT && ch * 8 >= kmain && ch * 8 < kdims ? tail + slot * tst + (ch * 8 - kmain)
                                                                                      : kb + slot * kst + (ch * 8 < kdims ? ch * 8 : 0);
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(ks + r * DP * 2 + ((ch ^ (r & 7)) << 4)), "l"(src), "r"(ch * 8 < kdims ? 16 : 0));
        }
        for (int i = threadIdx.x; i < KT * (VP / 8); i += 128) {
            const int r = i / (VP / 8), ch = i % (VP / 8);
            int slot = slot0 + min(r, key_hi - base);
            if (!EXPLICIT && slot >= cap) slot -= cap;
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(vs + r * VP * 2 + ((ch ^ (r & 7)) << 4)),
                         "l"(vb + slot * vst + (ch * 8 < vdims ? ch * 8 : 0)), "r"(ch * 8 < vdims ? 16 : 0));
        }
        asm volatile("cp.async.commit_group;\n" ::);
    };
    load_tile(key_lo, 0);

    const int qa = q_lo + warp * 16 + g, qb = qa + 8;
    const int pa = len + qa, pb = len + qb;  // positions of this thread's two rows
    uint32_t qf[DP / 16][4];
    {
        const __nv_bfloat16 *ra = q0 + (size_t)min(qa, a.S - 1) * a.q_stride;
        const __nv_bfloat16 *rb = q0 + (size_t)min(qb, a.S - 1) * a.q_stride;
#pragma unroll
        for (int ks = 0; ks < DP / 16; ++ks)
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                const int d = ks * 16 + h * 8 + 2 * c;
                const bool in = d < dim;
                qf[ks][2 * h] = in ? *reinterpret_cast<const uint32_t *>(ra + d) : 0u;
                qf[ks][2 * h + 1] = in ? *reinterpret_cast<const uint32_t *>(rb + d) : 0u;
            }
    }
    const float sl = a.scale * 1.44269504088896341f;  // scores in powers of two
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f}, o[VP / 8][4];
#pragma unroll
    for (int i = 0; i < VP / 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) o[i][j] = 0.f;
    const int w_first = len + q_lo + warp * 16, w_last = len + min(a.S - 1, q_lo + warp * 16 + 15);

    int buf = 0;
    for (int base = key_lo; base <= key_hi; base += KT, buf ^= 1) {
        const bool more = base + KT <= key_hi;
        if (more) load_tile(base + KT, buf ^ 1);
        if (more) asm volatile("cp.async.wait_group 1;\n" ::: "memory");
        else asm volatile("cp.async.wait_group 0;\n" ::: "memory");
        __syncthreads();
        const uint32_t ks0 = (uint32_t)__cvta_generic_to_shared(smem) + buf * (KB + VB), vs0 = ks0 + KB;
        if (base <= w_last && base + KT - 1 > w_first - window) {
            float s[8][4];
#pragma unroll
            for (int nt = 0; nt < 8; ++nt) {
#pragma unroll
                for (int j = 0; j < 4; ++j) s[nt][j] = 0.f;
                const int r = nt * 8 + (lane & 7);
#pragma unroll
                for (int k2 = 0; k2 < DP / 32; ++k2) {
                    uint32_t b0, b1, b2, b3;
                    const uint32_t addr = ks0 + r * DP * 2 + (((k2 * 4 + (lane >> 3)) ^ (r & 7)) << 4);
                    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                                 : "=r"(b0), "=r"(b1), "=r"(b2), "=r"(b3) : "r"(addr));
                    mma_bf16(s[nt], qf[2 * k2], b0, b1);
                    mma_bf16(s[nt], qf[2 * k2 + 1], b2, b3);
                }
            }
            const bool edge = base + KT - 1 > w_first || base <= w_last - window;
            float bm[2] = {-INFINITY, -INFINITY};
#pragma unroll
            for (int nt = 0; nt < 8; ++nt)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const int key = base + nt * 8 + 2 * c + (j & 1), p = j < 2 ? pa : pb;
                    float v = s[nt][j] * sl;
                    if (edge && (key > p || key <= p - window)) v = -INFINITY;
                    s[nt][j] = v;
                    bm[j >> 1] = fmaxf(bm[j >> 1], v);
                }
            float corr[2];
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                bm[h] = fmaxf(bm[h], __shfl_xor_sync(0xffffffffu, bm[h], 1));
                bm[h] = fmaxf(bm[h], __shfl_xor_sync(0xffffffffu, bm[h], 2));
                const float m_new = fmaxf(m_run[h], bm[h]);
                corr[h] = m_new == -INFINITY ? 1.f : exp2f(m_run[h] - m_new);
                m_run[h] = m_new;
                l_run[h] *= corr[h];
            }
#pragma unroll
            for (int nt = 0; nt < 8; ++nt)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const float m = m_run[j >> 1], p = m == -INFINITY ? 0.f : exp2f(s[nt][j] - m);
                    s[nt][j] = p;
                    l_run[j >> 1] += p;  // this thread's keys; the quad's shares are added at the end
                }
#pragma unroll
            for (int i = 0; i < VP / 8; ++i) { o[i][0] *= corr[0]; o[i][1] *= corr[0]; o[i][2] *= corr[1]; o[i][3] *= corr[1]; }
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) {
                uint32_t hi[4], lo[4];
                split_pair(s[2 * kk][0], s[2 * kk][1], hi[0], lo[0]);
                split_pair(s[2 * kk][2], s[2 * kk][3], hi[1], lo[1]);
                split_pair(s[2 * kk + 1][0], s[2 * kk + 1][1], hi[2], lo[2]);
                split_pair(s[2 * kk + 1][2], s[2 * kk + 1][3], hi[3], lo[3]);
                const int r = kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7);
#pragma unroll
                for (int vv = 0; vv < VP / 16; ++vv) {
                    uint32_t b0, b1, b2, b3;
                    const uint32_t addr = vs0 + r * VP * 2 + (((vv * 2 + (lane >> 4)) ^ (r & 7)) << 4);
                    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                                 : "=r"(b0), "=r"(b1), "=r"(b2), "=r"(b3) : "r"(addr));
                    mma_bf16(o[2 * vv], hi, b0, b1);
                    mma_bf16(o[2 * vv], lo, b0, b1);
                    mma_bf16(o[2 * vv + 1], hi, b2, b3);
                    mma_bf16(o[2 * vv + 1], lo, b2, b3);
                }
            }
        }
        __syncthreads();  // the tile is free for the load after next
    }
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 1);
        l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 2);
        const int qi = h ? qb : qa;
        if (qi >= a.S) continue;
        float inv = 1.f / l_run[h];
        if constexpr (EXPLICIT)
            if (a.gate) inv /= 1.f + expf(-__bfloat162float(a.gate[qi * a.gate_stride + head]));
        __nv_bfloat16 *dst = (__nv_bfloat16 *)a.out + ((size_t)rrow * a.S + qi) * out_stride + (size_t)head * a.vdim;
#pragma unroll
        for (int i = 0; i < VP / 8; ++i) {
            const int d = i * 8 + 2 * c;
            if (d < a.vdim)
                *reinterpret_cast<__nv_bfloat162 *>(dst + d) = __floats2bfloat162_rn(o[i][2 * h] * inv, o[i][2 * h + 1] * inv);
        }
    }
}

// ---------------------------------------------------------------------------
// Decode in bf16: one query per sequence, one launch.  The (up to 16) query heads of a KV head are the
// rows of the MMA, the keys its columns.  grid (nsplit, G * head groups, rows), 4 warps.
//   - The cached keys of the window are cut into nsplit runs; a CTA's warps deal its run out 16 at a time
//     and stream it through rings of their own in shared memory (cp.async, no CTA barrier in the loop).
//     The first of it is requested before the dependency wait: it belongs to earlier steps.
//   - Every CTA rotates and normalises its query heads; the last split also the new key, mixes the new
//     value, stores both in the cache and attends to them from shared memory.
//   - The warps meet in shared memory, the splits in the CTA that arrives last.
// ---------------------------------------------------------------------------
constexpr int WD_STAGES = 3;

template <int DP, int VP>
__global__ void __launch_bounds__(128) window_decode_mma_kernel(WindowAttnArgs a) {
    extern __shared__ __align__(1024) uint8_t smem[];
    constexpr int KB = 16 * DP * 2, VB = 16 * VP * 2, STAGE = KB + VB;
    __shared__ __align__(128) uint8_t fresh[STAGE];            // the new token's key and value as row 0 of a tile
    __shared__ __align__(16) __nv_bfloat16 qs[16][DP + 8];
    __shared__ float wm[4][16], wl[4][16];
    const KvLayer &l = a.kv.l;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, c = lane & 3;
    const int groups = (a.rep + 15) / 16, kvh = blockIdx.y / groups, hg = blockIdx.y % groups;
    const int head0 = kvh * a.rep + hg * 16, nh = min(16, a.rep - hg * 16);
    const int rrow = blockIdx.z, row = kv_row(a.kv, a.row0, rrow);
    const int pos = a.kv.lens[row], lo = max(0, pos - l.window + 1), n = pos - lo;  // cached keys in sight
    const int per = ((n + a.nsplit - 1) / a.nsplit + 63) & ~63;
    const int j0 = lo + (int)blockIdx.x * per, j1 = min(pos, j0 + per);
    const bool owns_new = (int)blockIdx.x == a.nsplit - 1;
    __nv_bfloat16 *kb = (__nv_bfloat16 *)l.k + ((size_t)row * l.kvh + kvh) * l.cap * l.kds;
    __nv_bfloat16 *vb = (__nv_bfloat16 *)l.v + ((size_t)row * l.kvh + kvh) * l.cap * l.vds;
    const uint32_t ring = (uint32_t)__cvta_generic_to_shared(smem) + warp * WD_STAGES * STAGE;
    const uint32_t fresh_s = (uint32_t)__cvta_generic_to_shared(fresh);

    auto load = [&](int base, int st) {
        if (base < j1) {
            const uint32_t ks = ring + st * STAGE, vs = ks + KB;
            const int slot0 = base % l.cap;
#pragma unroll
            for (int i = 0; i < 16 * (DP / 8) / 32; ++i) {
                const int idx = lane + 32 * i, r = idx / (DP / 8), ch = idx % (DP / 8);
                int slot = slot0 + min(r, j1 - 1 - base);  // keys past the run repeat its last (masked below)
                if (slot >= l.cap) slot -= l.cap;
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(ks + r * DP * 2 + ((ch ^ (r & 7)) << 4)),
                             "l"(kb + (size_t)slot * l.kds + (ch * 8 < l.kds ? ch * 8 : 0)), "r"(ch * 8 < l.kds ? 16 : 0));
            }
#pragma unroll
            for (int i = 0; i < 16 * (VP / 8) / 32; ++i) {
                const int idx = lane + 32 * i, r = idx / (VP / 8), ch = idx % (VP / 8);
                int slot = slot0 + min(r, j1 - 1 - base);
                if (slot >= l.cap) slot -= l.cap;
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(vs + r * VP * 2 + ((ch ^ (r & 7)) << 4)),
                             "l"(vb + (size_t)slot * l.vds + (ch * 8 < l.vds ? ch * 8 : 0)), "r"(ch * 8 < l.vds ? 16 : 0));
            }
        }
        asm volatile("cp.async.commit_group;\n" ::);  // one group per stage, also an empty one
    };
#pragma unroll
    for (int st = 0; st < WD_STAGES - 1; ++st) load(j0 + (st * 4 + warp) * 16, st);
    for (int i = threadIdx.x; i < STAGE / 16; i += 128) reinterpret_cast<uint4 *>(fresh)[i] = make_uint4(0u, 0u, 0u, 0u);
    for (int i = threadIdx.x; i < 16 * (DP + 8) / 8; i += 128) reinterpret_cast<uint4 *>(&qs[0][0])[i] = make_uint4(0u, 0u, 0u, 0u);
    __syncthreads();
    pdl_wait();
    pdl_launch_dependents();

    {
        const WindowPrepArgs &p = a.prep;
        const __nv_bfloat16 *tok = (const __nv_bfloat16 *)p.qkv + (size_t)rrow * p.stride;
        constexpr int NP = DP / 64;
        float u[NP], w[NP];
        for (int h = warp; h < nh; h += 4) {
            rotate_normalise<__nv_bfloat16, NP>(p, tok + (size_t)(head0 + h) * p.dim, pos, lane, u, w);
#pragma unroll
            for (int j = 0; j < NP; ++j)
                if (2 * (lane + 32 * j) < p.dim)
                    *reinterpret_cast<__nv_bfloat162 *>(&qs[h][2 * (lane + 32 * j)]) = __floats2bfloat162_rn(u[j], w[j]);
        }
        const int slot = pos % l.cap;
        if (owns_new && warp == 3) {
            rotate_normalise<__nv_bfloat16, NP>(p, tok + (size_t)(p.H + kvh) * p.dim, pos, lane, u, w);
#pragma unroll
            for (int j = 0; j < NP; ++j) {
                const int d = 2 * (lane + 32 * j);
                if (d >= p.dim) continue;
                const __nv_bfloat162 kv2 = __floats2bfloat162_rn(u[j], w[j]);
                *reinterpret_cast<__nv_bfloat162 *>(fresh + d * 2) = kv2;  // row 0: chunk order is the plain one
                if (hg == 0) *reinterpret_cast<__nv_bfloat162 *>(kb + (size_t)slot * l.kds + d) = kv2;
            }
        }
        if (owns_new && warp == 2) {
            const __nv_bfloat16 *src = tok + (size_t)(p.H + p.G) * p.dim + (size_t)kvh * p.vdim;
            __nv_bfloat16 *first = (__nv_bfloat16 *)p.v_first + ((size_t)rrow * p.G + kvh) * p.vdim;
            for (int d = lane; d < p.vdim; d += 32) {
                __nv_bfloat16 v = src[d];
                if (p.v_mode == 1 && hg == 0) first[d] = v;
                if (p.v_mode == 2) v = __float2bfloat16_rn((1.f - p.lambda) * __bfloat162float(v) + p.lambda * __bfloat162float(first[d]));
                *reinterpret_cast<__nv_bfloat16 *>(fresh + KB + d * 2) = v;
                if (hg == 0) vb[(size_t)slot * l.vds + d] = v;
            }
        }
    }
    __syncthreads();

    uint32_t qf[DP / 16][4];
#pragma unroll
    for (int ks = 0; ks < DP / 16; ++ks)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            qf[ks][2 * h] = *reinterpret_cast<const uint32_t *>(&qs[g][ks * 16 + h * 8 + 2 * c]);
            qf[ks][2 * h + 1] = *reinterpret_cast<const uint32_t *>(&qs[g + 8][ks * 16 + h * 8 + 2 * c]);
        }
    const float sl = a.scale * 1.44269504088896341f;  // scores in powers of two
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f}, o[VP / 8][4];
#pragma unroll
    for (int i = 0; i < VP / 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) o[i][j] = 0.f;

    // 16 keys in shared memory, the first `live` of which count
    auto attend = [&](uint32_t ks0, int live) {
        const uint32_t vs0 = ks0 + KB;
        float s[2][4], bm[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
#pragma unroll
            for (int j = 0; j < 4; ++j) s[nt][j] = 0.f;
            const int r = nt * 8 + (lane & 7);
#pragma unroll
            for (int k2 = 0; k2 < DP / 32; ++k2) {
                uint32_t b0, b1, b2, b3;
                const uint32_t addr = ks0 + r * DP * 2 + (((k2 * 4 + (lane >> 3)) ^ (r & 7)) << 4);
                asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                             : "=r"(b0), "=r"(b1), "=r"(b2), "=r"(b3) : "r"(addr));
                mma_bf16(s[nt], qf[2 * k2], b0, b1);
                mma_bf16(s[nt], qf[2 * k2 + 1], b2, b3);
            }
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                s[nt][j] = nt * 8 + 2 * c + (j & 1) < live ? s[nt][j] * sl : -INFINITY;
                bm[j >> 1] = fmaxf(bm[j >> 1], s[nt][j]);
            }
        }
        float corr[2];
#pragma unroll
        for (int h = 0; h < 2; ++h) {  // live > 0: the maximum is finite
            bm[h] = fmaxf(bm[h], __shfl_xor_sync(0xffffffffu, bm[h], 1));
            bm[h] = fmaxf(bm[h], __shfl_xor_sync(0xffffffffu, bm[h], 2));
            const float m_new = fmaxf(m_run[h], bm[h]);
            corr[h] = exp2f(m_run[h] - m_new);
            m_run[h] = m_new;
            l_run[h] *= corr[h];
        }
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                s[nt][j] = exp2f(s[nt][j] - m_run[j >> 1]);
                l_run[j >> 1] += s[nt][j];
            }
        uint32_t hi[4], lw[4];
        split_pair(s[0][0], s[0][1], hi[0], lw[0]);
        split_pair(s[0][2], s[0][3], hi[1], lw[1]);
        split_pair(s[1][0], s[1][1], hi[2], lw[2]);
        split_pair(s[1][2], s[1][3], hi[3], lw[3]);
#pragma unroll
        for (int i = 0; i < VP / 8; ++i) { o[i][0] *= corr[0]; o[i][1] *= corr[0]; o[i][2] *= corr[1]; o[i][3] *= corr[1]; }
        const int r = lane & 15;
#pragma unroll
        for (int vv = 0; vv < VP / 16; ++vv) {
            uint32_t b0, b1, b2, b3;
            const uint32_t addr = vs0 + r * VP * 2 + (((vv * 2 + (lane >> 4)) ^ (r & 7)) << 4);
            asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                         : "=r"(b0), "=r"(b1), "=r"(b2), "=r"(b3) : "r"(addr));
            mma_bf16(o[2 * vv], hi, b0, b1);
            mma_bf16(o[2 * vv], lw, b0, b1);
            mma_bf16(o[2 * vv + 1], hi, b2, b3);
            mma_bf16(o[2 * vv + 1], lw, b2, b3);
        }
    };

    int st = 0;
    for (int base = j0 + warp * 16; base < j1; base += 64) {
        load(base + (WD_STAGES - 1) * 64, (st + WD_STAGES - 1) % WD_STAGES);
        asm volatile("cp.async.wait_group %0;\n" ::"n"(WD_STAGES - 1) : "memory");
        __syncwarp();
        attend(ring + st * STAGE, j1 - base);
        // The products have consumed every matrix load of this stage (a tensor-core instruction waits for
        // its operands), so the refill at the top of the next pass cannot overtake them.
        __syncwarp();
        st = (st + 1) % WD_STAGES;
    }
    if (owns_new && warp == 0) attend(fresh_s, 1);
    asm volatile("cp.async.wait_group 0;\n" ::: "memory");
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 1);
        l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 2);
        if (c == 0) { wm[warp][g + 8 * h] = m_run[h]; wl[warp][g + 8 * h] = l_run[h]; }
    }
    __syncthreads();  // the rings are free: they take the warps' sums, [4][16][VP] floats
    float *wacc = reinterpret_cast<float *>(smem);
#pragma unroll
    for (int i = 0; i < VP / 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) wacc[((size_t)warp * 16 + g + 8 * (j >> 1)) * VP + i * 8 + 2 * c + (j & 1)] = o[i][j];
    __syncthreads();
    __nv_bfloat16 *out = (__nv_bfloat16 *)a.out + ((size_t)rrow * a.H + head0) * a.vdim;
    const size_t p0 = ((size_t)rrow * a.H + head0) * a.nsplit;
    for (int i = threadIdx.x; i < nh * a.vdim; i += 128) {
        const int hh = i / a.vdim, d = i % a.vdim;
        const float M = fmaxf(fmaxf(wm[0][hh], wm[1][hh]), fmaxf(wm[2][hh], wm[3][hh]));
        float L = 0.f, A = 0.f;
#pragma unroll
        for (int w = 0; w < 4; ++w) {
            const float e = wm[w][hh] == -INFINITY ? 0.f : exp2f(wm[w][hh] - M);
            L += e * wl[w][hh];
            A += e * wacc[((size_t)w * 16 + hh) * VP + d];
        }
        if (a.nsplit == 1) {
            out[i] = __float2bfloat16_rn(A / L);
        } else {
            const size_t pi = p0 + (size_t)hh * a.nsplit + blockIdx.x;
            a.part_acc[pi * a.vdim + d] = A;
            if (d == 0) { a.part_ml[pi * 2] = M; a.part_ml[pi * 2 + 1] = L; }
        }
    }
    if (a.nsplit == 1) return;
    // the CTA that arrives last merges the splits
    __shared__ int last;
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) {
        int *counter = a.counters + (size_t)rrow * gridDim.y + blockIdx.y;
        last = atomicAdd(counter, 1) == a.nsplit - 1;
        if (last) *counter = 0;  // at rest for the next launch
    }
    __syncthreads();
    if (!last) return;
    __threadfence();
    // split weights per head, normalised, in shared memory ([nh][nsplit] floats; nsplit <= 64)
    float *wt = reinterpret_cast<float *>(smem);
    for (int hh = warp; hh < nh; hh += 4) {
        const float *ml = a.part_ml + (p0 + (size_t)hh * a.nsplit) * 2;
        float m[2], ls[2], M = -INFINITY, L = 0.f;
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const int sp = lane + 32 * k;
            m[k] = sp < a.nsplit ? __ldcg(ml + sp * 2) : -INFINITY;
            ls[k] = sp < a.nsplit ? __ldcg(ml + sp * 2 + 1) : 0.f;
            M = fmaxf(M, m[k]);
        }
#pragma unroll
        for (int q = 16; q > 0; q >>= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, q));
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            m[k] = m[k] == -INFINITY ? 0.f : exp2f(m[k] - M);
            L = fmaf(m[k], ls[k], L);
        }
#pragma unroll
        for (int q = 16; q > 0; q >>= 1) L += __shfl_xor_sync(0xffffffffu, L, q);
#pragma unroll
        for (int k = 0; k < 2; ++k)
            if (lane + 32 * k < a.nsplit) wt[hh * a.nsplit + lane + 32 * k] = m[k] / L;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < nh * a.vdim; i += 128) {
        const int hh = i / a.vdim, d = i % a.vdim;
        const float *acc = a.part_acc + (p0 + (size_t)hh * a.nsplit) * a.vdim + d;
        float A = 0.f;
#pragma unroll 8
        for (int k = 0; k < a.nsplit; ++k) A = fmaf(wt[hh * a.nsplit + k], __ldcg(acc + (size_t)k * a.vdim), A);
        out[i] = __float2bfloat16_rn(A);
    }
}

template <int DP, int VP>
cudaError_t launch_decode(const WindowAttnArgs &a, dim3 grid, cudaStream_t s) {
    constexpr int smem = 4 * WD_STAGES * 16 * (DP + VP) * 2 > 4 * 16 * VP * 4 ? 4 * WD_STAGES * 16 * (DP + VP) * 2 : 4 * 16 * VP * 4;
    static bool configured[64] = {false};
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev >= 0 && dev < 64 && !configured[dev]) {
        cudaError_t e = cudaFuncSetAttribute(window_decode_mma_kernel<DP, VP>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) return e;
        configured[dev] = true;
    }
    return launch_kernel(window_decode_mma_kernel<DP, VP>, grid, dim3(128), (size_t)smem, s, a);
}

template <typename T, int REP>
cudaError_t launch_simt(const WindowAttnArgs &a, dim3 grid, size_t smem, cudaStream_t s) {
    if (a.vdim <= 32) return launch_kernel(window_attn_kernel<T, REP, 1>, grid, dim3(128), smem, s, a);
    if (a.vdim <= 64) return launch_kernel(window_attn_kernel<T, REP, 2>, grid, dim3(128), smem, s, a);
    if (a.vdim <= 128) return launch_kernel(window_attn_kernel<T, REP, 4>, grid, dim3(128), smem, s, a);
    return launch_kernel(window_attn_kernel<T, REP, 8>, grid, dim3(128), smem, s, a);
}

template <int DP, int VP, class Args>
cudaError_t launch_mma(const Args &a, int heads, int nrows, cudaStream_t s) {
    constexpr int smem = 2 * 64 * (DP + VP) * 2;
    static bool configured[64] = {false};
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev >= 0 && dev < 64 && !configured[dev]) {
        cudaError_t e = cudaFuncSetAttribute(window_attn_mma_kernel<DP, VP, Args>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) return e;
        configured[dev] = true;
    }
    return launch_kernel(window_attn_mma_kernel<DP, VP, Args>, dim3((a.S + 63) / 64, heads, nrows), dim3(128), (size_t)smem, s, a);
}

template <typename T>
int launch_window(const ab2_kv *kv, WindowAttnArgs a, int nrows, int max_len, cudaStream_t s) {
    cudaError_t e;
    const KvLayer &l = a.kv.l;
    const bool on_mma = sizeof(T) == 2 && a.dim % 8 == 0 && a.vdim % 8 == 0 && a.dim <= 128 && a.vdim <= 128 && a.q_stride % 2 == 0;
    if (!(on_mma && a.S == 1)) {
        const dim3 pgrid((a.H + 2 * a.prep.G + 7) / 8, a.S, nrows);
        e = launch_kernel(window_prep_kernel<T>, pgrid, dim3(256), 0, s, a.prep);
        if (e != cudaSuccess) return fail(AB2_ERR_CUDA, "window preparation launch failed: %s", cudaGetErrorString(e));
    }
    if (on_mma && a.S >= 16) {
        if (a.dim <= 64) e = a.vdim <= 64 ? launch_mma<64, 64>(a, a.H, nrows, s) : launch_mma<64, 128>(a, a.H, nrows, s);
        else e = a.vdim <= 64 ? launch_mma<128, 64>(a, a.H, nrows, s) : launch_mma<128, 128>(a, a.H, nrows, s);
        if (e != cudaSuccess) return fail(AB2_ERR_CUDA, "window attention launch failed: %s", cudaGetErrorString(e));
        return AB2_OK;
    }
    if (on_mma && a.S == 1) {
        const int units = l.kvh * ((a.rep + 15) / 16) * nrows, reach = std::min(l.window, max_len);
        // two CTAs per SM hold the streams that cover HBM's latency; a split keeps at least 128 keys
        const int want = (2 * device_sm_count() + units - 1) / units;
        a.nsplit = std::max(1, std::min(std::min(want, (reach + 127) / 128), kv->max_splits));
        const dim3 grid(a.nsplit, l.kvh * ((a.rep + 15) / 16), nrows);
        if (a.dim <= 64) e = a.vdim <= 64 ? launch_decode<64, 64>(a, grid, s) : launch_decode<64, 128>(a, grid, s);
        else e = a.vdim <= 64 ? launch_decode<128, 64>(a, grid, s) : launch_decode<128, 128>(a, grid, s);
        if (e != cudaSuccess) return fail(AB2_ERR_CUDA, "window attention launch failed: %s", cudaGetErrorString(e));
        return AB2_OK;
    }
    const int REPS = a.rep == 1 ? 1 : a.rep == 2 ? 2 : a.rep <= 4 ? 4 : 8;
    const int groups = (a.rep + REPS - 1) / REPS, units = l.kvh * groups * nrows;
    a.nsplit = 1;
    if (a.S == 1) {
        const int reach = std::min(l.window, max_len), want = (2 * device_sm_count() + units - 1) / units;
        a.nsplit = std::max(1, std::min(std::min(want, (reach + 127) / 128), kv->max_splits));
    }
    dim3 grid(a.nsplit, l.kvh * groups, nrows * a.S);
    const size_t smem = ((size_t)REPS * l.kds + 4 * (size_t)REPS * a.vdim) * 4;
    if (REPS == 1) e = launch_simt<T, 1>(a, grid, smem, s);
    else if (REPS == 2) e = launch_simt<T, 2>(a, grid, smem, s);
    else if (REPS == 4) e = launch_simt<T, 4>(a, grid, smem, s);
    else e = launch_simt<T, 8>(a, grid, smem, s);
    if (e == cudaSuccess && a.nsplit > 1)
        e = launch_kernel(window_merge_kernel<T>, dim3(a.H, nrows), dim3(std::min(128, (a.vdim + 31) / 32 * 32)), 0, s, a);
    if (e != cudaSuccess) return fail(AB2_ERR_CUDA, "window attention launch failed: %s", cudaGetErrorString(e));
    return AB2_OK;
}

}  // namespace

int window_attention(const ab2_kv *kv, WindowAttnArgs a, int nrows, int max_len, ab2_dtype dtype, cudaStream_t s) {
    a.part_acc = kv->part_acc; a.part_ml = kv->part_ml; a.counters = kv->counters;
    return dtype == AB2_F32 ? launch_window<float>(kv, a, nrows, max_len, s) : launch_window<__nv_bfloat16>(kv, a, nrows, max_len, s);
}

bool prompt_attention_serves(int dim, int tail, int vdim) {
    return dim % 8 == 0 && tail % 8 == 0 && vdim % 8 == 0 && dim + tail <= 192 && vdim <= 128;
}

int prompt_attention(const PromptAttnArgs &a, cudaStream_t s) {
    if (prompt_tc_serves(a)) return prompt_tc_attention(a, s);
    const int d = a.dim + a.tail_dims;
    cudaError_t e;
    if (d <= 64) e = a.vdim <= 64 ? launch_mma<64, 64>(a, a.heads, 1, s) : launch_mma<64, 128>(a, a.heads, 1, s);
    else if (d <= 128) e = a.vdim <= 64 ? launch_mma<128, 64>(a, a.heads, 1, s) : launch_mma<128, 128>(a, a.heads, 1, s);
    else e = a.vdim <= 64 ? launch_mma<192, 64>(a, a.heads, 1, s) : launch_mma<192, 128>(a, a.heads, 1, s);
    if (e != cudaSuccess) return fail(AB2_ERR_CUDA, "prompt attention launch failed: %s", cudaGetErrorString(e));
    return AB2_OK;
}

}  // namespace ab2
