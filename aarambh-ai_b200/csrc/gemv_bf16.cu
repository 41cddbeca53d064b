// Decode linears over dense bf16 weights: HBM-bound streaming on the warp-level tensor cores.
//
// A CTA owns 16 weight rows (with a gated unit: 8 gate rows and the 8 matching up rows) and its 8 warps
// deal out K in chunks of 32 columns.  Per chunk a lane reads 16 bytes of row g, 16 of row g + 8
// and 16 of each of its tokens (g = lane / 4; lane % 4 picks the 8 columns), which are two
// mma.sync.m16n8k16 fragments as they stand: the same permutation of K on both operands leaves the
// dot product alone.  Weights are the rows of the MMA, up to 8 * NT tokens its columns; the warps'
// sums meet in shared memory.  The first weights are requested before the dependency wait.
// The grouped modes run one CTA column per active expert and walk that expert's pairs; a batch of
// weights (one per head) runs one grid layer each.
#include <algorithm>

#include "linear_bf16.cuh"

using namespace ab2;

namespace ab2 {
namespace {

constexpr int GV_WARPS = 8, GV_UNROLL = 4;

__device__ __forceinline__ uint4 ld_stream(const __nv_bfloat16 *p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];\n" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

template <int MODE, int NT>
__global__ void __launch_bounds__(GV_WARPS * 32) gemv_bf16_kernel(LinArgs a) {
    constexpr bool GROUPED = MODE == LIN_MOE_GLU || MODE == LIN_MOE_DOWN, DUAL = MODE == LIN_MOE_GLU || MODE == LIN_GLU;
    constexpr int TOK = 8 * NT;
    __shared__ float red[GV_WARPS][TOK][17];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, c = lane & 3;
    const int nch = (a.K + 31) >> 5;
    const uint4 zero = make_uint4(0u, 0u, 0u, 0u);

    int r0 = 0, cnt = a.M, tile0 = blockIdx.y * TOK, tile_step = gridDim.y * TOK;
    size_t wbase = 0;
    if (GROUPED) {
        pdl_wait();
        pdl_launch_dependents();
        if ((int)blockIdx.y >= a.r.active[0]) return;
        const int e = a.r.active[1 + blockIdx.y];
        r0 = a.r.offset[e];
        cnt = a.r.offset[e + 1] - r0;
        wbase = (size_t)e * a.N * a.K;
        tile0 = 0; tile_step = TOK;
    }
    if (MODE == LIN_DENSE) wbase = (size_t)blockIdx.z * a.wb;
    const int n0 = blockIdx.x * (DUAL ? 8 : 16);
    const __nv_bfloat16 *wa = a.w + wbase + (size_t)min(n0 + g, a.N - 1) * a.K + c * 8;
    const __nv_bfloat16 *wb = DUAL ? a.w2 + wbase + (size_t)min(n0 + g, a.N - 1) * a.K + c * 8
                                                  : a.w + wbase + (size_t)min(n0 + g + 8, a.N - 1) * a.K + c * 8;
    uint4 va[GV_UNROLL], vb[GV_UNROLL];
    auto load_w = [&](int ch0) {
#pragma unroll
        for (int u = 0; u < GV_UNROLL; ++u) {
            const int ch = ch0 + u * GV_WARPS;
            const bool ok = ch * 32 + c * 8 < a.K;  // K is a multiple of 8
            va[u] = ok ? ld_stream(wa + ch * 32) : zero;
            vb[u] = ok ? ld_stream(wb + ch * 32) : zero;
        }
    };
    load_w(warp);
    if (!GROUPED) {
        pdl_wait();
        pdl_launch_dependents();
    }
    const __nv_bfloat16 *x = (const __nv_bfloat16 *)a.x + (MODE == LIN_DENSE ? blockIdx.z * a.xb : 0);
    const size_t ldx = MODE == LIN_DENSE ? a.ldx : a.K;
    for (int m0 = tile0; m0 < cnt; m0 += tile_step) {
        const __nv_bfloat16 *xp[NT];
        bool xv[NT];
#pragma unroll
        for (int j = 0; j < NT; ++j) {
            const int m = m0 + j * 8 + g;
            xv[j] = m < cnt;
            const int mm = xv[j] ? m : cnt - 1;
            const int row = MODE == LIN_MOE_GLU ? a.r.perm[r0 + mm] / a.r.top : r0 + mm;
            xp[j] = x + row * ldx + c * 8;
        }
        float acc[NT][4];
#pragma unroll
        for (int j = 0; j < NT; ++j)
#pragma unroll
            for (int i = 0; i < 4; ++i) acc[j][i] = 0.f;
        for (int ch0 = warp; ch0 < nch; ch0 += GV_WARPS * GV_UNROLL) {
            if (!(m0 == tile0 && ch0 == warp)) load_w(ch0);
#pragma unroll
            for (int u = 0; u < GV_UNROLL; ++u) {
                const int ch = ch0 + u * GV_WARPS;
                const bool ok = ch * 32 + c * 8 < a.K;
#pragma unroll
                for (int j = 0; j < NT; ++j) {
                    const uint4 b = ok && xv[j] ? *reinterpret_cast<const uint4 *>(xp[j] + ch * 32) : zero;
                    mma_bf16(acc[j], va[u].x, vb[u].x, va[u].y, vb[u].y, b.x, b.y);
                    mma_bf16(acc[j], va[u].z, vb[u].z, va[u].w, vb[u].w, b.z, b.w);
                }
            }
        }
#pragma unroll
        for (int j = 0; j < NT; ++j) {
            red[warp][j * 8 + 2 * c][g] = acc[j][0];
            red[warp][j * 8 + 2 * c + 1][g] = acc[j][1];
            red[warp][j * 8 + 2 * c][g + 8] = acc[j][2];
            red[warp][j * 8 + 2 * c + 1][g + 8] = acc[j][3];
        }
        __syncthreads();
        constexpr int ROWS = DUAL ? 8 : 16;
        for (int i = threadIdx.x; i < ROWS * TOK; i += GV_WARPS * 32) {
            const int row = i % ROWS, t = i / ROWS, m = m0 + t, n = n0 + row;
            if (m >= cnt || n >= a.N) continue;
            float v = 0.f, v2 = 0.f;
#pragma unroll
            for (int w = 0; w < GV_WARPS; ++w) {
                v += red[w][t][row];
                if (DUAL) v2 += red[w][t][row + 8];
            }
            if (DUAL) {
                const float s = MODE == LIN_MOE_GLU && a.scored ? a.r.score[a.r.perm[r0 + m]] : 1.f;
                ((__nv_bfloat16 *)a.y)[(size_t)(r0 + m) * a.N + n] = __float2bfloat16_rn(glu_value(a.glu, s * v, s * v2, a.limit));
            } else if (MODE == LIN_MOE_DOWN) {
                ((float *)a.y)[(size_t)a.r.perm[r0 + m] * a.N + n] = a.out_scale * v;
            } else {
                const size_t o = blockIdx.z * a.yb + m * a.ldy + n;
                if (a.epi == LIN_F32) ((float *)a.y)[o] = softcap_value(v, a.cap);
                else {
                    if (a.epi == LIN_ACT) v = lin_act_value(v, n < a.act_n);
                    if (a.epi == LIN_GATE) v *= lin_act_value(__bfloat162float(((const __nv_bfloat16 *)a.gate)[m * a.gate_ld + blockIdx.z]), false);
                    ((__nv_bfloat16 *)a.y)[o] = __float2bfloat16_rn(v);
                }
            }
        }
        __syncthreads();
    }
}

template <int MODE>
cudaError_t launch_gemv(const LinArgs &a, cudaStream_t s) {
    constexpr bool GROUPED = MODE == LIN_MOE_GLU || MODE == LIN_MOE_DOWN;
    const int rows = MODE == LIN_MOE_GLU || MODE == LIN_GLU ? 8 : 16;
    // most pairs one expert can get: every token once
    const int m = GROUPED ? a.r.pairs / a.r.top : a.M;
    const int nt = m <= 8 ? 1 : m <= 16 ? 2 : 4;
    dim3 grid((a.N + rows - 1) / rows, GROUPED ? std::min(a.r.E, a.r.pairs) : (m + 8 * nt - 1) / (8 * nt), MODE == LIN_DENSE ? a.batch : 1);
    if (nt == 1) return launch_kernel(gemv_bf16_kernel<MODE, 1>, grid, dim3(GV_WARPS * 32), 0, s, a);
    if (nt == 2) return launch_kernel(gemv_bf16_kernel<MODE, 2>, grid, dim3(GV_WARPS * 32), 0, s, a);
    return launch_kernel(gemv_bf16_kernel<MODE, 4>, grid, dim3(GV_WARPS * 32), 0, s, a);
}

}  // namespace

int gemv_bf16(const LinArgs &a, int mode, cudaStream_t s) {
    cudaError_t e = mode == LIN_DENSE     ? launch_gemv<LIN_DENSE>(a, s)
                    : mode == LIN_MOE_GLU ? launch_gemv<LIN_MOE_GLU>(a, s)
                    : mode == LIN_GLU     ? launch_gemv<LIN_GLU>(a, s)
                                          : launch_gemv<LIN_MOE_DOWN>(a, s);
    if (e != cudaSuccess) return fail(AB2_ERR_CUDA, "bf16 GEMV launch failed: %s", cudaGetErrorString(e));
    return AB2_OK;
}

}  // namespace ab2
