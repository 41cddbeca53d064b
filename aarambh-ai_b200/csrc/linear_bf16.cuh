// Linear layers over dense bf16 weights, plain or grouped by expert (internal header).
//
// Three kernels serve them: a streaming GEMV for a few tokens (gemv_bf16.cu), a tcgen05 GEMM for
// many (gemm_bf16_tc.cu) and a tiled CUDA-core kernel for f32 activations and odd shapes
// (linear_simt.cu), each in four modes.
#pragma once

#include "common.cuh"

namespace ab2 {

// What becomes of the f32 sum of a plain linear.
enum LinEpilogue : int {
    LIN_STORE = 0,  // rounded to the activation type
    LIN_F32 = 1,    // stored as f32
    LIN_ACT = 2,    // silu for output channels below act_n, sigmoid from there on; activation type
    LIN_GATE = 3    // times the sigmoid of one gate value per row (and weight, see LinArgs::batch); activation type
};

enum LinMode : int {
    LIN_DENSE = 0,     // y[m] = x[m] . W^T
    LIN_MOE_GLU = 1,   // act[r] = glu(s (x_t . Wg_e^T), s (x_t . Wu_e^T)), r a sorted (token, expert) pair
    LIN_MOE_DOWN = 2,  // y[pair] = out_scale (act[r] . Wd_e^T), f32
    LIN_GLU = 3        // act[m] = glu(x[m] . Wg^T, x[m] . Wu^T)
};

// Gated units.
enum GluKind : int {
    GLU_CLAMPED = 0,   // g = min(gate, limit), u = clamp(up, -limit, limit): g sigmoid(1.702 g) (u + 1)
    GLU_SILU = 1       // gate sigmoid(gate) up
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
    const __nv_bfloat16 *w2;  // LIN_MOE_GLU, LIN_GLU: the up weights
    const void *x;
    void *y;
    int N, K, M;              // N rows per expert in the grouped modes; M rows of x
    long long ldx, ldy;       // LIN_DENSE: row strides of x and y in elements
    int epi, act_n;
    float cap;                // LIN_F32: the sum z becomes cap tanh(z / cap); 0: stays z
    int glu;                  // GluKind
    float limit;              // clamp of the gated unit
    float out_scale;          // LIN_MOE_DOWN
    bool scored;              // LIN_MOE_GLU: r.score multiplies the gate and up products
    MoeRoute r;
    // LIN_DENSE over several weights of one shape (one per head): weight b reads x + b * xb and writes
    // y + b * yb; weight b starts at w + b * wb
    int batch;
    long long wb, xb, yb;
    const void *gate;         // LIN_GATE: gate[m * gate_ld + b] in the activation type
    long long gate_ld;
};

__device__ __forceinline__ float glu_value(int kind, float gate, float up, float limit) {
    if (kind == GLU_SILU) return __fdividef(gate, 1.f + __expf(-gate)) * up;
    const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
    return __fdividef(g, 1.f + __expf(-1.702f * g)) * (u + 1.f);
}
__device__ __forceinline__ float glu_value_exact(int kind, float gate, float up, float limit) {
    if (kind == GLU_SILU) return gate / (1.f + expf(-gate)) * up;
    const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
    return g / (1.f + expf(-1.702f * g)) * (u + 1.f);
}
__device__ __forceinline__ float softcap_value(float z, float cap) { return cap > 0.f ? cap * tanhf(z / cap) : z; }
__device__ __forceinline__ float lin_act_value(float v, bool silu) {
    const float sg = 1.f / (1.f + expf(-v));
    return silu ? v * sg : sg;
}

// y = epilogue(x . W^T) for a FMT_BF16 weight
int linear_bf16(const ab2_qweight *w, const void *x, int M, ab2_dtype dtype, void *y, int epi, int act_n, cudaStream_t s);
// The same with the arguments filled in by the caller (strides, batches of weights, other epilogues).
int linear_dense(const LinArgs &a, ab2_dtype dtype, cudaStream_t s);
// act [M][ff] = glu(x Wg^T, x Wu^T) for every token
int linear_glu(const ab2_qweight *gate, const ab2_qweight *up, const void *x, int M, ab2_dtype dtype, void *act, int glu, float limit, cudaStream_t s);
// The two grouped linears of a mixture of experts.  x [T][K] and act [pairs][ff] in the activation
// type, y [pairs][width] f32; `gathered` is scratch for pairs x K activations.
int linear_moe_glu(const ab2_qweight *gate, const ab2_qweight *up, const void *x, ab2_dtype dtype, void *act, int glu, float limit,
                   bool scored, const MoeRoute &r, void *gathered, cudaStream_t s);
int linear_moe_down(const ab2_qweight *down, const void *act, ab2_dtype dtype, float *y, float out_scale, const MoeRoute &r, cudaStream_t s);

// kernel families
int linear_simt(const LinArgs &a, int mode, ab2_dtype dtype, cudaStream_t s);
int gemv_bf16(const LinArgs &a, int mode, cudaStream_t s);
int gemm_bf16_tc(const LinArgs &a, int mode, cudaStream_t s);

}  // namespace ab2
