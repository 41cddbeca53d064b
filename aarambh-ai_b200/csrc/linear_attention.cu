// Lightning attention: linear attention with a fixed decay per head.  Per head
//   S_t = d S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t
// with S [dim][vdim] in f32, kept per (layer, sequence) in the cache.  A sequence whose length is 0
// starts from zero whatever its slot held before.
//
//   lightning_serial_kernel   token by token, f32 on CUDA cores: decode, f32 models, any head size
#include <algorithm>

#include "stack.cuh"

using namespace ab2;

namespace ab2 {
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
    cudaError_t e = dtype == AB2_F32 ? launch_serial<float>(a, nrows, s) : launch_serial<__nv_bfloat16>(a, nrows, s);
    if (e != cudaSuccess) return fail(AB2_ERR_CUDA, "lightning attention launch failed: %s", cudaGetErrorString(e));
    return AB2_OK;
}

}  // namespace ab2
