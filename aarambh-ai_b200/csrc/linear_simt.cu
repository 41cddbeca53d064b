// Dense-weight linears on CUDA cores with f32 arithmetic: every activation type and shape.  The
// path of f32 models (true 32-bit products) and of shapes whose rows do not start on 16 bytes.
// Also the selection among the three kernel families.
#include <algorithm>

#include "linear_bf16.cuh"

using namespace ab2;

namespace ab2 {
int device_sm_count();
namespace {

constexpr int TM = 64, TN = 64, TK = 16;

// One CTA: TM rows x TN channels, 4 x 4 per thread.  blockIdx.z is the expert (grouped modes) or the
// weight of a batch.
template <typename T, int MODE>
__global__ void __launch_bounds__(256) linear_simt_kernel(LinArgs a) {
    constexpr bool GROUPED = MODE == LIN_MOE_GLU || MODE == LIN_MOE_DOWN, DUAL = MODE == LIN_MOE_GLU || MODE == LIN_GLU;
    __shared__ float xs[TK][TM + 4], ws[TK][TN + 4], us[DUAL ? TK : 1][TN + 4];
    __shared__ int xrow[TM];
    pdl_wait();
    pdl_launch_dependents();
    const int n0 = blockIdx.x * TN, e = blockIdx.z;
    int r0 = 0, cnt = a.M;
    if (GROUPED) { r0 = a.r.offset[e]; cnt = a.r.offset[e + 1] - r0; }
    const int m0 = blockIdx.y * TM;
    if (m0 >= cnt) return;
    const size_t wbase = GROUPED ? (size_t)e * a.N * a.K : MODE == LIN_DENSE ? (size_t)e * a.wb : 0;
    const T *x = (const T *)a.x + (MODE == LIN_DENSE ? e * a.xb : 0);
    const size_t ldx = MODE == LIN_DENSE ? a.ldx : a.K;
    for (int i = threadIdx.x; i < TM; i += 256) {
        const int m = m0 + i;
        xrow[i] = m >= cnt ? -1 : MODE == LIN_MOE_GLU ? a.r.perm[r0 + m] / a.r.top : r0 + m;
    }
    __syncthreads();
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4], acc2[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = acc2[i][j] = 0.f;
    for (int k0 = 0; k0 < a.K; k0 += TK) {
        for (int i = threadIdx.x; i < TM * TK; i += 256) {
            const int m = i / TK, k = i % TK;
            xs[k][m] = (xrow[m] >= 0 && k0 + k < a.K) ? to_f32(x[xrow[m] * ldx + k0 + k]) : 0.f;
        }
        for (int i = threadIdx.x; i < TN * TK; i += 256) {
            const int n = i / TK, k = i % TK;
            const bool ok = n0 + n < a.N && k0 + k < a.K;
            const size_t idx = wbase + (size_t)(n0 + n) * a.K + k0 + k;
            ws[k][n] = ok ? __bfloat162float(a.w[idx]) : 0.f;
            if (DUAL) us[k][n] = ok ? __bfloat162float(a.w2[idx]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < TK; ++k) {
            float xv[4], wv[4], uv[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) { xv[i] = xs[k][ty * 4 + i]; wv[i] = ws[k][tx * 4 + i]; if (DUAL) uv[i] = us[k][tx * 4 + i]; }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    acc[i][j] = fmaf(xv[i], wv[j], acc[i][j]);
                    if (DUAL) acc2[i][j] = fmaf(xv[i], uv[j], acc2[i][j]);
                }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int m = m0 + ty * 4 + i;
        if (m >= cnt) continue;
        const int pair = GROUPED ? a.r.perm[r0 + m] : 0;
        const float s = MODE == LIN_MOE_GLU && a.scored ? a.r.score[pair] : 1.f;
        const float gate = MODE == LIN_DENSE && a.epi == LIN_GATE ? lin_act_value(to_f32(((const T *)a.gate)[m * a.gate_ld + e]), false) : 1.f;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int n = n0 + tx * 4 + j;
            if (n >= a.N) continue;
            const float v = acc[i][j];
            if (DUAL) {
                ((T *)a.y)[(size_t)(r0 + m) * a.N + n] = from_f32<T>(glu_value_exact(a.glu, s * v, s * acc2[i][j], a.limit));
            } else if (MODE == LIN_MOE_DOWN) {
                ((float *)a.y)[(size_t)pair * a.N + n] = a.out_scale * v;
            } else {
                const size_t o = e * a.yb + m * a.ldy + n;
                if (a.epi == LIN_F32) ((float *)a.y)[o] = softcap_value(v, a.cap);
                else ((T *)a.y)[o] = from_f32<T>(a.epi == LIN_ACT ? lin_act_value(v, n < a.act_n) : v * gate);
            }
        }
    }
}

template <typename T>
cudaError_t launch_simt(const LinArgs &a, int mode, cudaStream_t s) {
    const bool grouped = mode == LIN_MOE_GLU || mode == LIN_MOE_DOWN;
    const int rows = grouped ? a.r.pairs / a.r.top : a.M;  // an expert gets a token once
    dim3 grid((a.N + TN - 1) / TN, (rows + TM - 1) / TM, grouped ? a.r.E : mode == LIN_DENSE ? a.batch : 1);
    if (mode == LIN_GLU) return launch_kernel(linear_simt_kernel<T, LIN_GLU>, grid, dim3(256), 0, s, a);
    if (mode == LIN_DENSE) return launch_kernel(linear_simt_kernel<T, LIN_DENSE>, grid, dim3(256), 0, s, a);
    if (mode == LIN_MOE_GLU) return launch_kernel(linear_simt_kernel<T, LIN_MOE_GLU>, grid, dim3(256), 0, s, a);
    return launch_kernel(linear_simt_kernel<T, LIN_MOE_DOWN>, grid, dim3(256), 0, s, a);
}

// Rows of the decode GEMV: beyond this many the tensor-memory GEMM's token tiles pay.
constexpr int GEMV_MAX_ROWS = 32;

bool rows_aligned(const void *w, const void *x, int K) { return K % 8 == 0 && (((uintptr_t)w | (uintptr_t)x) & 15) == 0; }

// Copies the activations of every sorted pair next to each other: out[r] = x[perm[r] / top].
__global__ void gather_pairs_kernel(const __nv_bfloat16 *x, __nv_bfloat16 *out, const int *perm, int top, int K) {
    pdl_wait();
    pdl_launch_dependents();
    const uint4 *src = reinterpret_cast<const uint4 *>(x + (size_t)(perm[blockIdx.x] / top) * K);
    uint4 *dst = reinterpret_cast<uint4 *>(out + (size_t)blockIdx.x * K);
    for (int i = threadIdx.x; i < K / 8; i += blockDim.x) dst[i] = src[i];
}

}  // namespace

int linear_simt(const LinArgs &a, int mode, ab2_dtype dtype, cudaStream_t s) {
    cudaError_t e;
    switch (dtype) {
    case AB2_F32: e = launch_simt<float>(a, mode, s); break;
    case AB2_F16: e = launch_simt<__half>(a, mode, s); break;
    default: e = launch_simt<__nv_bfloat16>(a, mode, s); break;
    }
    if (e != cudaSuccess) return fail(AB2_ERR_CUDA, "linear launch failed: %s", cudaGetErrorString(e));
    return AB2_OK;
}

int linear_dense(const LinArgs &a, ab2_dtype dtype, cudaStream_t s) {
    if (dtype != AB2_BF16 || !rows_aligned(a.w, a.x, a.K) || a.ldx % 8 != 0 || a.xb % 8 != 0 || a.wb % 8 != 0) return linear_simt(a, LIN_DENSE, dtype, s);
    return a.M <= GEMV_MAX_ROWS || a.batch > 1 || a.epi == LIN_GATE ? gemv_bf16(a, LIN_DENSE, s) : gemm_bf16_tc(a, LIN_DENSE, s);
}

int linear_bf16(const ab2_qweight *w, const void *x, int M, ab2_dtype dtype, void *y, int epi, int act_n, cudaStream_t s) {
    LinArgs a = {};
    a.w = (const __nv_bfloat16 *)w->codes; a.x = x; a.y = y; a.N = w->N; a.K = w->K; a.M = M; a.epi = epi; a.act_n = act_n;
    a.ldx = a.K; a.ldy = a.N; a.batch = 1;
    return linear_dense(a, dtype, s);
}

int linear_glu(const ab2_qweight *gate, const ab2_qweight *up, const void *x, int M, ab2_dtype dtype, void *act, int glu, float limit, cudaStream_t s) {
    LinArgs a = {};
    a.w = (const __nv_bfloat16 *)gate->codes; a.w2 = (const __nv_bfloat16 *)up->codes; a.x = x; a.y = act;
    a.N = gate->N; a.K = gate->K; a.M = M; a.glu = glu; a.limit = limit;
    if (dtype != AB2_BF16 || !rows_aligned(a.w, x, a.K)) return linear_simt(a, LIN_GLU, dtype, s);
    return M <= GEMV_MAX_ROWS ? gemv_bf16(a, LIN_GLU, s) : gemm_bf16_tc(a, LIN_GLU, s);
}

int linear_moe_glu(const ab2_qweight *gate, const ab2_qweight *up, const void *x, ab2_dtype dtype, void *act, int glu, float limit,
                   bool scored, const MoeRoute &r, void *gathered, cudaStream_t s) {
    LinArgs a = {};
    a.w = (const __nv_bfloat16 *)gate->codes; a.w2 = (const __nv_bfloat16 *)up->codes; a.x = x; a.y = act;
    a.N = gate->N / r.E; a.K = gate->K; a.M = r.pairs / r.top; a.glu = glu; a.limit = limit; a.scored = scored; a.r = r;
    if (dtype != AB2_BF16 || !rows_aligned(a.w, x, a.K)) return linear_simt(a, LIN_MOE_GLU, dtype, s);
    if (r.pairs <= 2 * GEMV_MAX_ROWS) return gemv_bf16(a, LIN_MOE_GLU, s);
    cudaError_t e = launch_kernel(gather_pairs_kernel, dim3(r.pairs), dim3(std::min(256, std::max(32, a.K / 8))), 0, s,
                                  (const __nv_bfloat16 *)x, (__nv_bfloat16 *)gathered, (const int *)r.perm, r.top, a.K);
    if (e != cudaSuccess) return fail(AB2_ERR_CUDA, "gather launch failed: %s", cudaGetErrorString(e));
    a.x = gathered; a.M = r.pairs;
    return gemm_bf16_tc(a, LIN_MOE_GLU, s);
}

int linear_moe_down(const ab2_qweight *down, const void *act, ab2_dtype dtype, float *y, float out_scale, const MoeRoute &r, cudaStream_t s) {
    LinArgs a = {};
    a.w = (const __nv_bfloat16 *)down->codes; a.x = act; a.y = y;
    a.N = down->N / r.E; a.K = down->K; a.M = r.pairs; a.out_scale = out_scale; a.r = r;
    if (dtype != AB2_BF16 || !rows_aligned(a.w, act, a.K)) return linear_simt(a, LIN_MOE_DOWN, dtype, s);
    return r.pairs <= 2 * GEMV_MAX_ROWS ? gemv_bf16(a, LIN_MOE_DOWN, s) : gemm_bf16_tc(a, LIN_MOE_DOWN, s);
}

}  // namespace ab2
