// Lightning attention: linear attention with a fixed decay per head.  Per head
//   S_t = d S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t
// with S [dim][vdim] in f32, kept per (layer, sequence) in the cache.  A sequence whose length is 0
// starts from zero whatever its slot held before.
//
//   lightning_serial_kernel   token by token, f32 on CUDA cores: decode, f32 models, any head size
//   lightning_chunk_kernel    prompts in bf16, 64 tokens at a time on the warp-level tensor cores:
//                             with i, j counted inside the chunk and S the state before it
//                                 o_i   = d^(i+1) S^T q_i + sum_{j <= i} d^(i-j) (q_i . k_j) v_j
//                                 S_new = d^n S + sum_j d^(n-1-j) k_j v_j^T
//
// Where the heads of a prompt leave SMs idle it is cut into segments of whole chunks that run side by
// side: a first launch (SUMS) forms every segment's own sum  sum_j d^(L-1-j) k_j v_j^T  (L the segment
// length) and copies the state before the prompt, a second (lightning_scan_kernel) makes the state before
// each segment of them,  S_(r+1) = d^L S_r + sum_r,  and the third computes the outputs.
//
// q, k and v are bf16 as the projections leave them; everything else of the recurrence is f32.
// Where an f32 quantity is an operand of a tensor-core product (the state, the decayed scores, the
// decayed keys) it goes in as two bf16 terms, the rounded value and what rounding left, so the
// products carry it to about 16 significant bits; the state itself is accumulated in f32.
#include <algorithm>

#include "stack.cuh"

using namespace ab2;

namespace ab2 {
int device_sm_count();
namespace {

// grid (ceil(vdim / 32), H, rows), 8 warps.  A lane owns a value column, a warp DPW key rows of S,
// in registers.
template <typename T, int DPW>
__global__ void __launch_bounds__(256) lightning_serial_kernel(LightningArgs a) {
    constexpr int DIMP = 8 * DPW;
    constexpr int TB = DPW == 32 ? 8 : 16;  // tokens staged in shared memory at a time
    __shared__ __align__(16) float2 kq[TB][DIMP];
    __shared__ float vs[TB][32], red[TB][8][33];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int head = blockIdx.y, v0 = blockIdx.x * 32, vcol = v0 + lane;
    pdl_wait();
    pdl_launch_dependents();
    const int rrow = blockIdx.z, row = kv_row(a.kv, a.row0, rrow);
    float *state = a.kv.l.state + ((size_t)row * a.H + head) * a.dim * a.vdim;
    const float decay = a.decay_pow[(size_t)head * (LIGHTNING_CHUNK + 1) + 1];
    const bool fresh = a.kv.lens[row] == 0;
    float S[DPW];
#pragma unroll
    for (int i = 0; i < DPW; ++i) {
        const int d = warp * DPW + i;
        S[i] = !fresh && d < a.dim && vcol < a.vdim ? state[(size_t)d * a.vdim + vcol] : 0.f;
    }
    const T *base = (const T *)a.qkv + (size_t)rrow * a.S * a.stride;
    const size_t koff = (size_t)a.H * a.dim, voff = 2 * koff;
    for (int t0 = 0; t0 < a.S; t0 += TB) {
        const int nt = min(TB, a.S - t0);
        for (int i = threadIdx.x; i < nt * DIMP; i += 256) {
            const int t = i / DIMP, d = i % DIMP;
            const T *r = base + (size_t)(t0 + t) * a.stride + (size_t)head * a.dim + d;
            kq[t][d] = d < a.dim ? make_float2(to_f32(r[koff]), to_f32(r[0])) : make_float2(0.f, 0.f);
        }
        for (int i = threadIdx.x; i < nt * 32; i += 256) {
            const int t = i >> 5, j = i & 31;
            vs[t][j] = v0 + j < a.vdim ? to_f32(base[(size_t)(t0 + t) * a.stride + voff + (size_t)head * a.vdim + v0 + j]) : 0.f;
        }
        __syncthreads();
        for (int t = 0; t < nt; ++t) {
            const float v = vs[t][lane];
            float o = 0.f;
#pragma unroll
            for (int i = 0; i < DPW; i += 2) {
                const float4 p = *reinterpret_cast<const float4 *>(&kq[t][warp * DPW + i]);
                S[i] = fmaf(p.x, v, decay * S[i]);
                o = fmaf(S[i], p.y, o);
                S[i + 1] = fmaf(p.z, v, decay * S[i + 1]);
                o = fmaf(S[i + 1], p.w, o);
            }
            red[t][warp][lane] = o;
        }
        __syncthreads();
        for (int i = threadIdx.x; i < nt * 32; i += 256) {
            const int t = i >> 5, j = i & 31;
            float o = 0.f;
#pragma unroll
            for (int w = 0; w < 8; ++w) o += red[t][w][j];
            if (v0 + j < a.vdim) a.out[((size_t)rrow * a.S + t0 + t) * a.H * a.vdim + (size_t)head * a.vdim + v0 + j] = o;
        }
        // the next block's staging may start: it touches kq / vs, which every warp has left, and red is
        // written again only after the next barrier
    }
#pragma unroll
    for (int i = 0; i < DPW; ++i) {
        const int d = warp * DPW + i;
        if (d < a.dim && vcol < a.vdim) state[(size_t)d * a.vdim + vcol] = S[i];
    }
}

__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4t(uint32_t addr, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void split_pair(float x, float y, uint32_t &hi, uint32_t &lo) {
    const __nv_bfloat16 xh = __float2bfloat16_rn(x), yh = __float2bfloat16_rn(y);
    const __nv_bfloat16 xl = __float2bfloat16_rn(x - __bfloat162float(xh)), yl = __float2bfloat16_rn(y - __bfloat162float(yh));
    hi = (uint32_t)__bfloat16_as_ushort(xh) | ((uint32_t)__bfloat16_as_ushort(yh) << 16);
    lo = (uint32_t)__bfloat16_as_ushort(xl) | ((uint32_t)__bfloat16_as_ushort(yl) << 16);
}
// Byte offset of 16-byte chunk `ch` of row `r` in a tile of `cols` bf16 columns, placed so that the
// eight rows of a matrix load fall on different banks.
template <int COLS>
__device__ __forceinline__ uint32_t tile_off(int r, int ch) {
    if (COLS == 32) return r * 64 + ((ch ^ ((r >> 1) & 3)) << 4);
    return r * COLS * 2 + ((ch ^ (r & 7)) << 4);
}

// grid (ceil(vdim / VS), H, rows), 4 warps.  A warp owns 16 tokens of the chunk's outputs and DP / 4 key
// rows of the state's slice of VS value columns (accumulators in registers for the whole prompt; a
// two-term copy in shared memory feeds the next chunk's product with the queries).
template <int DP, int VS, bool SUMS>
__global__ void __launch_bounds__(128) lightning_chunk_kernel(LightningArgs a) {
    constexpr int C = LIGHTNING_CHUNK, MT = DP / 64, NV = VS / 8;
    constexpr int QB = C * DP * 2, VB = C * VS * 2, SB = DP * VS * 2, STAGE = 2 * QB + VB;
    extern __shared__ __align__(1024) uint8_t smem[];
    __shared__ float pw[C + 1];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, c = lane & 3;
    const int head = blockIdx.y, v0 = blockIdx.x * VS;
    const uint32_t sm = (uint32_t)__cvta_generic_to_shared(smem), s_hi = sm + 2 * STAGE, s_lo = s_hi + SB;
    for (int i = threadIdx.x; i <= C; i += 128) pw[i] = a.decay_pow[(size_t)head * (C + 1) + i];
    pdl_wait();
    pdl_launch_dependents();
    const int rrow = blockIdx.z / a.segs, seg = blockIdx.z % a.segs, row = kv_row(a.kv, a.row0, rrow);
    const int seg0 = seg * a.seg_len, S_len = min(a.seg_len, a.S - seg0);  // tokens of this CTA
    float *state = a.kv.l.state + ((size_t)row * a.H + head) * a.dim * a.vdim;
    // scratch slots: from SUMS segment r's own sum (r < segs - 1) and the state before the prompt (the last),
    // after lightning_scan_kernel the state before segment r
    const size_t slot_elems = (size_t)a.H * a.dim * a.vdim;
    float *slots = a.scratch + (size_t)rrow * a.segs * slot_elems + (size_t)head * a.dim * a.vdim;
    const bool fresh = a.kv.lens[row] == 0;
    const __nv_bfloat16 *base = (const __nv_bfloat16 *)a.qkv + ((size_t)rrow * a.S + seg0) * a.stride;
    const __nv_bfloat16 *qb = base + (size_t)head * a.dim, *kb = qb + (size_t)a.H * a.dim;
    const __nv_bfloat16 *vb = base + 2 * (size_t)a.H * a.dim + (size_t)head * a.vdim + v0;

    auto load = [&](int t0, int buf) {
        const uint32_t q = sm + buf * STAGE, k = q + QB, v = k + QB;
        for (int i = threadIdx.x; i < C * (DP / 8); i += 128) {
            const int r = i / (DP / 8), ch = i % (DP / 8);
            const bool in = t0 + r < S_len && ch * 8 < a.dim;  // what is not there is zero
            const size_t off = in ? (size_t)(t0 + r) * a.stride + ch * 8 : 0;
            const uint32_t d = tile_off<DP>(r, ch);
            if (!SUMS) asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(q + d), "l"(qb + off), "r"(in ? 16 : 0));
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(k + d), "l"(kb + off), "r"(in ? 16 : 0));
        }
        for (int i = threadIdx.x; i < C * (VS / 8); i += 128) {
            const int r = i / (VS / 8), ch = i % (VS / 8);
            const bool in = t0 + r < S_len && v0 + ch * 8 < a.vdim;
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(v + tile_off<VS>(r, ch)),
                         "l"(vb + (in ? (size_t)(t0 + r) * a.stride + ch * 8 : 0)), "r"(in ? 16 : 0));
        }
        asm volatile("cp.async.commit_group;\n" ::);
    };
    const bool copies = SUMS && seg == a.segs - 1;  // this CTA hands on the state before the prompt
    if (!copies) load(0, 0);

    float S[MT][NV][4];  // key rows (warp * MT + mt) * 16 + g, + 8; value columns n * 8 + 2c, + 1
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int n = 0; n < NV; ++n)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int d = (warp * MT + mt) * 16 + g + (j >> 1) * 8, v = v0 + n * 8 + 2 * c + (j & 1);
                const bool in = d < a.dim && v < a.vdim;
                const size_t at = (size_t)d * a.vdim + v;
                if (SUMS) S[mt][n][j] = copies && !fresh && in ? state[at] : 0.f;
                else if (a.segs == 1) S[mt][n][j] = !fresh && in ? state[at] : 0.f;
                else S[mt][n][j] = in ? slots[(size_t)seg * slot_elems + at] : 0.f;
            }
    auto publish = [&]() {
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
            for (int n = 0; n < NV; ++n)
#pragma unroll
                for (int h = 0; h < 2; ++h) {
                    uint32_t hi, lo;
                    split_pair(S[mt][n][2 * h], S[mt][n][2 * h + 1], hi, lo);
                    const uint32_t off = tile_off<VS>((warp * MT + mt) * 16 + g + h * 8, n) + 4 * c;
                    asm volatile("st.shared.u32 [%0], %1;\n" ::"r"(s_hi + off), "r"(hi) : "memory");
                    asm volatile("st.shared.u32 [%0], %1;\n" ::"r"(s_lo + off), "r"(lo) : "memory");
                }
    };
    if (!SUMS) publish();

    int buf = 0;
    for (int t0 = 0; t0 < (copies ? 0 : S_len); t0 += C, buf ^= 1) {
        const int n_tok = min(C, S_len - t0);
        asm volatile("cp.async.wait_group 0;\n" ::: "memory");
        __syncthreads();  // this chunk's tiles and the state's copy are visible; the other buffers are free
        if (t0 + C < S_len) load(t0 + C, buf ^ 1);
        const uint32_t qs = sm + buf * STAGE, ks = qs + QB, vs = ks + QB;

        if constexpr (!SUMS) {
        uint32_t qf[DP / 16][4];
#pragma unroll
        for (int k = 0; k < DP / 16; ++k) ldsm4(qs + tile_off<DP>(warp * 16 + (lane & 15), k * 2 + (lane >> 4)), qf[k]);
        const int i0 = warp * 16 + g, i1 = i0 + 8;
        float o[NV][4];
#pragma unroll
        for (int n = 0; n < NV; ++n)
#pragma unroll
            for (int j = 0; j < 4; ++j) o[n][j] = 0.f;
        // S^T q of the state before the chunk
#pragma unroll
        for (int k = 0; k < DP / 16; ++k)
#pragma unroll
            for (int n2 = 0; n2 < NV / 2; ++n2) {
                uint32_t b[4];
                const uint32_t off = tile_off<VS>(k * 16 + (lane & 15), n2 * 2 + (lane >> 4));
                ldsm4t(s_hi + off, b);
                mma_bf16(o[2 * n2], qf[k], b[0], b[1]);
                mma_bf16(o[2 * n2 + 1], qf[k], b[2], b[3]);
                ldsm4t(s_lo + off, b);
                mma_bf16(o[2 * n2], qf[k], b[0], b[1]);
                mma_bf16(o[2 * n2 + 1], qf[k], b[2], b[3]);
            }
        const float d0 = pw[i0 + 1], d1 = pw[i1 + 1];
#pragma unroll
        for (int n = 0; n < NV; ++n) { o[n][0] *= d0; o[n][1] *= d0; o[n][2] *= d1; o[n][3] *= d1; }
        // tokens of the chunk up to the query, 16 at a time
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
            if (kk > warp) break;
            float s[2][4];
#pragma unroll
            for (int h = 0; h < 2; ++h) {
#pragma unroll
                for (int j = 0; j < 4; ++j) s[h][j] = 0.f;
#pragma unroll
                for (int k2 = 0; k2 < DP / 32; ++k2) {
                    uint32_t b[4];
                    ldsm4(ks + tile_off<DP>(kk * 16 + h * 8 + (lane & 7), k2 * 4 + (lane >> 3)), b);
                    mma_bf16(s[h], qf[2 * k2], b[0], b[1]);
                    mma_bf16(s[h], qf[2 * k2 + 1], b[2], b[3]);
                }
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const int dist = (j < 2 ? i0 : i1) - (kk * 16 + h * 8 + 2 * c + (j & 1));
                    s[h][j] = dist >= 0 ? s[h][j] * pw[dist] : 0.f;
                }
            }
            uint32_t hi[4], lo[4];
            split_pair(s[0][0], s[0][1], hi[0], lo[0]);
            split_pair(s[0][2], s[0][3], hi[1], lo[1]);
            split_pair(s[1][0], s[1][1], hi[2], lo[2]);
            split_pair(s[1][2], s[1][3], hi[3], lo[3]);
#pragma unroll
            for (int n2 = 0; n2 < NV / 2; ++n2) {
                uint32_t b[4];
                ldsm4t(vs + tile_off<VS>(kk * 16 + (lane & 15), n2 * 2 + (lane >> 4)), b);
                mma_bf16(o[2 * n2], hi, b[0], b[1]);
                mma_bf16(o[2 * n2 + 1], hi, b[2], b[3]);
                mma_bf16(o[2 * n2], lo, b[0], b[1]);
                mma_bf16(o[2 * n2 + 1], lo, b[2], b[3]);
            }
        }
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            const int i = h ? i1 : i0;
            if (i >= n_tok) continue;
            float *dst = a.out + ((size_t)rrow * a.S + seg0 + t0 + i) * a.H * a.vdim + (size_t)head * a.vdim + v0;
#pragma unroll
            for (int n = 0; n < NV; ++n)
                if (v0 + n * 8 + 2 * c < a.vdim) *reinterpret_cast<float2 *>(dst + n * 8 + 2 * c) = make_float2(o[n][2 * h], o[n][2 * h + 1]);
        }
        }
        // the state after the chunk
        const float dn = pw[n_tok];
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
            for (int n = 0; n < NV; ++n)
#pragma unroll
                for (int j = 0; j < 4; ++j) S[mt][n][j] *= dn;
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
            uint32_t vf[NV / 2][4];
#pragma unroll
            for (int n2 = 0; n2 < NV / 2; ++n2) ldsm4t(vs + tile_off<VS>(kk * 16 + (lane & 15), n2 * 2 + (lane >> 4)), vf[n2]);
            float f[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int back = n_tok - 1 - (kk * 16 + (j >> 1) * 8 + 2 * c + (j & 1));
                f[j] = back >= 0 ? pw[back] : 0.f;
            }
#pragma unroll
            for (int mt = 0; mt < MT; ++mt) {
                uint32_t r[4], hi[4], lo[4];
                ldsm4t(ks + tile_off<DP>(kk * 16 + (lane >> 4) * 8 + (lane & 7), (warp * MT + mt) * 2 + ((lane >> 3) & 1)), r);
#pragma unroll
                for (int j = 0; j < 4; ++j)
                    split_pair(__uint_as_float(r[j] << 16) * f[(j >> 1) * 2], __uint_as_float(r[j] & 0xffff0000u) * f[(j >> 1) * 2 + 1], hi[j], lo[j]);
#pragma unroll
                for (int n2 = 0; n2 < NV / 2; ++n2) {
                    mma_bf16(S[mt][2 * n2], hi, vf[n2][0], vf[n2][1]);
                    mma_bf16(S[mt][2 * n2 + 1], hi, vf[n2][2], vf[n2][3]);
                    mma_bf16(S[mt][2 * n2], lo, vf[n2][0], vf[n2][1]);
                    mma_bf16(S[mt][2 * n2 + 1], lo, vf[n2][2], vf[n2][3]);
                }
            }
        }
        __syncthreads();  // every warp has read the state's copy
        if (!SUMS) publish();
    }
    if (!SUMS && seg != a.segs - 1) return;
    float *end = SUMS ? slots + (size_t)seg * slot_elems : state;
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int n = 0; n < NV; ++n)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int d = (warp * MT + mt) * 16 + g + (j >> 1) * 8, v = v0 + n * 8 + 2 * c + (j & 1);
                if (d < a.dim && v < a.vdim) end[(size_t)d * a.vdim + v] = S[mt][n][j];
            }
}

template <int DP, int VS, bool SUMS>
cudaError_t launch_chunk(const LightningArgs &a, int nrows, cudaStream_t s) {
    constexpr int smem = 2 * (2 * LIGHTNING_CHUNK * DP * 2 + LIGHTNING_CHUNK * VS * 2) + 2 * DP * VS * 2;
    static bool configured[64] = {false};
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev >= 0 && dev < 64 && !configured[dev]) {
        cudaError_t e = cudaFuncSetAttribute(lightning_chunk_kernel<DP, VS, SUMS>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) return e;
        configured[dev] = true;
    }
    return launch_kernel(lightning_chunk_kernel<DP, VS, SUMS>, dim3((a.vdim + VS - 1) / VS, a.H, nrows * a.segs), dim3(128), (size_t)smem, s, a);
}

// grid (blocks over a head's state, H, rows): the slots of one state element, in order.
__global__ void __launch_bounds__(256) lightning_scan_kernel(LightningArgs a) {
    pdl_wait();
    pdl_launch_dependents();
    const int n = a.dim * a.vdim, i = blockIdx.x * 256 + threadIdx.x;
    if (i >= n) return;
    float *slot = a.scratch + (size_t)blockIdx.z * a.segs * a.H * n + (size_t)blockIdx.y * n + i;
    const size_t step = (size_t)a.H * n;
    const float dl = powf(a.decay_pow[(size_t)blockIdx.y * (LIGHTNING_CHUNK + 1) + LIGHTNING_CHUNK], (float)(a.seg_len / LIGHTNING_CHUNK));
    float v[LIGHTNING_MAX_SEGMENTS];
#pragma unroll
    for (int r = 0; r < LIGHTNING_MAX_SEGMENTS; ++r) v[r] = r < a.segs ? slot[r * step] : 0.f;
    float S = 0.f;
#pragma unroll
    for (int r = 0; r < LIGHTNING_MAX_SEGMENTS; ++r)
        if (r == a.segs - 1) S = v[r];
#pragma unroll
    for (int r = 0; r < LIGHTNING_MAX_SEGMENTS; ++r) {
        if (r < a.segs) slot[r * step] = S;
        S = fmaf(dl, S, v[r]);
    }
}

template <int DP, int VS>
cudaError_t launch_prompt(const LightningArgs &a, int nrows, cudaStream_t s) {
    if (a.segs > 1) {
        cudaError_t e = launch_chunk<DP, VS, true>(a, nrows, s);
        if (e == cudaSuccess)
            e = launch_kernel(lightning_scan_kernel, dim3((a.dim * a.vdim + 255) / 256, a.H, nrows), dim3(256), 0, s, a);
        if (e != cudaSuccess) return e;
    }
    return launch_chunk<DP, VS, false>(a, nrows, s);
}

template <int DP>
cudaError_t launch_prompt(LightningArgs a, int nrows, cudaStream_t s) {
    // value slices of 64 columns, narrower ones while they leave SMs idle; then segments of at least four
    // chunks, until there are two CTAs per SM
    const int sms = device_sm_count();
    auto ctas = [&](int vs) { return (a.vdim + vs - 1) / vs * a.H * nrows; };
    const bool narrow = a.vdim <= 32 || (a.S < 8 * LIGHTNING_CHUNK && ctas(64) < sms);
    int segs = std::min(LIGHTNING_MAX_SEGMENTS / std::max(1, nrows), std::min((2 * sms) / ctas(narrow ? 32 : 64), a.S / (4 * LIGHTNING_CHUNK)));
    if (!a.scratch || segs < 2) segs = 1;
    a.seg_len = ((a.S + segs - 1) / segs + LIGHTNING_CHUNK - 1) / LIGHTNING_CHUNK * LIGHTNING_CHUNK;
    a.segs = (a.S + a.seg_len - 1) / a.seg_len;
    return narrow ? launch_prompt<DP, 32>(a, nrows, s) : launch_prompt<DP, 64>(a, nrows, s);
}

// Prompts whose heads fit the chunk kernel; a handful of tokens is quicker one by one.
bool chunk_eligible(const LightningArgs &a) {
    return a.S >= 16 && a.dim % 8 == 0 && a.vdim % 8 == 0 && a.dim <= 128 && a.stride % 8 == 0;
}

template <typename T>
cudaError_t launch_serial(const LightningArgs &a, int nrows, cudaStream_t s) {
    const dim3 grid((a.vdim + 31) / 32, a.H, nrows);
    if (a.dim <= 32) return launch_kernel(lightning_serial_kernel<T, 4>, grid, dim3(256), 0, s, a);
    if (a.dim <= 64) return launch_kernel(lightning_serial_kernel<T, 8>, grid, dim3(256), 0, s, a);
    if (a.dim <= 128) return launch_kernel(lightning_serial_kernel<T, 16>, grid, dim3(256), 0, s, a);
    return launch_kernel(lightning_serial_kernel<T, 32>, grid, dim3(256), 0, s, a);
}

}  // namespace

int lightning_attention(const LightningArgs &a, int nrows, ab2_dtype dtype, cudaStream_t s) {
    cudaError_t e;
    if (dtype == AB2_F32) e = launch_serial<float>(a, nrows, s);
    else if (!chunk_eligible(a)) e = launch_serial<__nv_bfloat16>(a, nrows, s);
    else e = a.dim <= 64 ? launch_prompt<64>(a, nrows, s) : launch_prompt<128>(a, nrows, s);
    if (e != cudaSuccess) return fail(AB2_ERR_CUDA, "lightning attention launch failed: %s", cudaGetErrorString(e));
    return AB2_OK;
}

}  // namespace ab2
