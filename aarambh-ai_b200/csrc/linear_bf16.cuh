// Linear layers over dense bf16 weights, plain or grouped by expert (internal header).
//
// Three kernels serve them: a streaming GEMV for a few tokens (gemv_bf16.cu), a tcgen05 GEMM for
// many (gemm_bf16_tc.cu) and a tiled CUDA-core kernel for f32 activations and odd shapes
// (linear_simt.cu), each in three modes.
#pragma once

#include "common.cuh"

namespace ab2 {

// What becomes of the f32 sum of a plain linear.
enum LinEpilogue : int {
    LIN_STORE = 0,  // rounded to the activation type
    LIN_F32 = 1,    // stored as f32
    LIN_ACT = 2     // silu for output channels below act_n, sigmoid from there on; activation type
};

enum LinMode : int {
    LIN_DENSE = 0,     // y[m] = x[m] . W^T
    LIN_MOE_GLU = 1,   // act[r] = glu(s (x_t . Wg_e^T), s (x_t . Wu_e^T)), r a sorted (token, expert) pair
    LIN_MOE_DOWN = 2   // y[pair] = act[r] . Wd_e^T, f32
};

// Routing of T tokens to `top` of E experts each.  Pair p = token * top + slot; the pairs are
// sorted by expert, expert e owning sorted positions [offset[e], offset[e + 1]).
struct MoeRoute {
    int E, top, pairs;
    int *offset;    // [E + 1]
    int *perm;      // [pairs] sorted position -> pair
    float *score;   // [pairs] by pair
    int *expert;    // [pairs] by pair
    int *active;    // [E + 1]: number of experts with at least one pair, then those experts
};

struct LinArgs {
    const __nv_bfloat16 *w;   // [N][K]; grouped: [E * N][K], the gate weights in LIN_MOE_GLU
    const __nv_bfloat16 *w2;  // LIN_MOE_GLU: the up weights
    const void *x;
    void *y;
    int N, K, M;              // N rows per expert in the grouped modes; M rows of x
    int epi, act_n;
    float limit;              // clamp of the gated unit
    MoeRoute r;
};

// g = min(gate, limit), u = clamp(up, -limit, limit): g sigmoid(1.702 g) (u + 1)
__device__ __forceinline__ float clamped_glu_value(float gate, float up, float limit) {
    const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
    return __fdividef(g, 1.f + __expf(-1.702f * g)) * (u + 1.f);
}
__device__ __forceinline__ float clamped_glu_value_exact(float gate, float up, float limit) {
    const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
    return g / (1.f + expf(-1.702f * g)) * (u + 1.f);
}
__device__ __forceinline__ float lin_act_value(float v, bool silu) {
    const float sg = 1.f / (1.f + expf(-v));
    return silu ? v * sg : sg;
}

// y = epilogue(x . W^T) for a FMT_BF16 weight
int linear_bf16(const ab2_qweight *w, const void *x, int M, ab2_dtype dtype, void *y, int epi, int act_n, cudaStream_t s);
// The two grouped linears of a mixture of experts.  x [T][K] and act [pairs][ff] in the activation
// type, y [pairs][width] f32; `gathered` is scratch for pairs x K activations.
int linear_moe_glu(const ab2_qweight *gate, const ab2_qweight *up, const void *x, ab2_dtype dtype, void *act, float limit,
                   const MoeRoute &r, void *gathered, cudaStream_t s);
int linear_moe_down(const ab2_qweight *down, const void *act, ab2_dtype dtype, float *y, const MoeRoute &r, cudaStream_t s);

// kernel families
int linear_simt(const LinArgs &a, int mode, ab2_dtype dtype, cudaStream_t s);
int gemv_bf16(const LinArgs &a, int mode, cudaStream_t s);
int gemm_bf16_tc(const LinArgs &a, int mode, cudaStream_t s);

}  // namespace ab2
