// Layer stacks: the parts shared by the mechanisms and the model (internal header).
#pragma once

#include <vector>

#include "common.cuh"
#include "kv_cache.cuh"
#include "linear_bf16.cuh"

namespace ab2 {

// ---- sliding-window attention (attention_window.cu) -----------------------------
struct WindowPrepArgs {
    KvLayerView kv;
    void *qkv;             // [nrows * S][stride]: H query heads, G key heads, G value heads; queries are rewritten
    long long stride;
    int S, row0, H, G, dim, vdim, rot_dims, qk_norm;
    const float *cos_t, *sin_t;  // [positions][rot_dims / 2]
    float eps;
    void *v_first;         // [nrows * S][G * vdim]
    int v_mode;            // 0 values as they are, 1 also keep them in v_first, 2 mix them with v_first
    float lambda;
};
struct WindowAttnArgs {
    WindowPrepArgs prep;   // one token per row in bf16: done inside the attention kernel
    KvLayerView kv;
    const void *q;         // head h of token t at t * q_stride + h * dim
    long long q_stride;
    void *out;             // [nrows * S][H * vdim]
    int S, row0, H, rep, dim, vdim, nsplit;
    float scale;
    float *part_acc, *part_ml;
    int *counters;         // [rows][G * head groups] split-arrival counters, 0 at rest
};
// Rotation, normalisation and value mixing of S new tokens per row, which are stored in the cache, and
// their attention; max_len bounds the rows' lengths with them.  `a.prep` and `a` name the same tokens.
int window_attention(const ab2_kv *kv, WindowAttnArgs a, int nrows, int max_len, ab2_dtype dtype, cudaStream_t s);

// ---- lightning attention (linear_attention.cu) ------------------------------------
struct LightningArgs {
    KvLayerView kv;
    const void *qkv;       // [nrows * S][stride]: q, k (heads x dim), v (heads x vdim), activated
    long long stride;
    float *out;            // [nrows * S][heads * vdim]
    int S, row0, H, dim, vdim;
    const float *decay_pow;  // [heads][LIGHTNING_CHUNK + 1]: powers 0, 1, ... of the head's decay
    float *scratch;          // states of a prompt's segments: LIGHTNING_MAX_SEGMENTS x heads x dim x vdim, or null
    int seg_len, segs;       // filled in by lightning_attention
};
constexpr int LIGHTNING_CHUNK = 64;
constexpr int LIGHTNING_MAX_SEGMENTS = 16;  // over all rows of a call
int lightning_attention(const LightningArgs &a, int nrows, ab2_dtype dtype, cudaStream_t s);

// ---- latent attention (attention_latent.cu) ----------------------------------------
// Keys and values of all heads are projections of one cached latent per token, plus one rotated key
// part that the heads share.  The cache row of a token is [latent (rank) | rotated part (rot)].
struct LatentArgs {
    KvLayerView kv;
    void *proj;            // [nrows * S][stride]: queries, heads x (dim + rot) | latent (rank) | key part (rot) | gates (heads)
    long long stride;
    int S, row0, H, dim, rot, rank, vdim, gated;
    const float *norm_w;   // [rank]
    float eps, scale;
    const float *cos_t, *sin_t;    // [positions][rot / 2]
    const __nv_bfloat16 *ukv;      // [H][dim key rows, vdim value rows][rank]
    const __nv_bfloat16 *absorb;   // [H][rank][dim]: the key rows transposed
    void *out;             // [nrows * S][H * vdim]
    void *work;            // latent_workspace bytes
    size_t work_bytes;
    float *part_acc, *part_ml;     // filled in by latent_attention
    int nsplit;
};
size_t latent_workspace(int H, int dim, int rot, int rank, int vdim, int tokens, int positions, ab2_dtype dtype);
// Norm and rotation of S new tokens per row, which are stored in the cache, and their attention; max_len
// bounds the rows' lengths with them.
int latent_attention(const ab2_kv *kv, LatentArgs a, int nrows, int max_len, ab2_dtype dtype, cudaStream_t s);
// absorb[h][r][d] = ukv[h][d][r] over the key rows
int latent_absorb_weights(const __nv_bfloat16 *ukv, __nv_bfloat16 *absorb, int H, int dim, int vdim, int rank, cudaStream_t s);
// The bf16 kernel of attention in the latent space (attention_latent_tc.cu): qx [nrows * S][H][kds] to
// ox [nrows * S][H][rank], or with a.nsplit > 1, which it chooses, to the splits' sums in a.part_acc, a.part_ml.
bool latent_tc_serves(int rank, int kds);
int latent_tc_attention(LatentArgs &a, const __nv_bfloat16 *qx, __nv_bfloat16 *ox, int cache_rows, int nrows, int max_len, cudaStream_t s);
constexpr int LATENT_ROWS = 32;    // (token, head) rows of a CTA of the decode kernel
constexpr int LATENT_PART_TILES = 320;  // row tiles x splits that the cache's scratch holds
static inline size_t latent_part_bytes(const ab2_layer_spec &sp) { return (size_t)LATENT_PART_TILES * LATENT_ROWS * sp.kv_rank * 4; }
static inline size_t latent_part_ml_bytes() { return (size_t)LATENT_PART_TILES * LATENT_ROWS * 2 * 4; }

// Causal attention of a prompt portion's S queries of one sequence over keys and values laid out
// position by position; the last `tail_dims` dimensions of a key are shared by the heads
// (bf16 only: on tcgen05 where the shape allows it, else window_attn_mma_kernel).
struct PromptAttnArgs {
    const __nv_bfloat16 *q, *k, *tail, *v, *gate;   // gate: [S][gate_stride] per head, or null
    long long q_stride, k_stride, tail_stride, v_stride, gate_stride, out_stride;  // between positions
    int k_head, v_head;    // between heads; a query head is dim + tail_dims elements
    __nv_bfloat16 *out;    // head h at h * vdim
    int S, heads, first, dim, tail_dims, vdim;   // `first`: position of the first query
    float scale;
};
bool prompt_attention_serves(int dim, int tail, int vdim);
bool prompt_tc_serves(const PromptAttnArgs &a);   // attention_prompt_tc.cu
int prompt_tc_attention(const PromptAttnArgs &a, cudaStream_t s);
int prompt_attention(const PromptAttnArgs &a, cudaStream_t s);

// ---- normalisation around the f32 residual stream (ops.cu) -------------------------
// Every form computes RMSNorm(v; w) of one row v per token.
enum ResidualNorm : int {
    RN_EMBED = 0,  // v = table[ids[t]];            x = norm
    RN_ADD = 1,    // v = sum of the token's parts; x += norm
    RN_FINAL = 2,  // v = x[t * step + step - 1];   out = norm
    RN_GATED = 3   // v = parts[t];                 out = norm * gate[t]
};
struct ResidualNormArgs {
    const float *w;
    float eps;
    int d;
    const __nv_bfloat16 *table;
    const uint32_t *ids;
    int vocab;
    const float *parts;    // RN_ADD: [T][nparts][d], RN_GATED: [T][d]
    int nparts, step;
    const void *gate;      // activation type, row stride gate_stride
    long long gate_stride;
    float *x;              // [T][d]
    void *out;             // activation type; RN_EMBED / RN_ADD: the new x rounded to it (null: not wanted)
    // RN_EMBED (whose w may be null: no norm) and RN_ADD, each null where it is not wanted
    const float *w_next;   // out is RMSNorm(x; w_next) of the new x
    const float *extra;    // RN_ADD: [T][d], one more part
    float *x0;             // RN_EMBED: [T][d], receives the embedding; RN_ADD: added to x
    const float *add;      // [d] vector added to x
};
int launch_residual_norm(const ResidualNormArgs &a, int mode, int rows, ab2_dtype dtype, cudaStream_t s);

// Activation of a feed-forward without a gate: out = a N(z) + b N(z^2) + c N(z^3) + e per row of n values, powers
// element by element, N the division by the root mean square over the row (ops.cu).
struct PolyNormArgs {
    const void *z;         // [rows][n], activation type
    void *out;
    int n;
    float a, b, c, e, eps;
};
int launch_poly_norm(const PolyNormArgs &p, int rows, ab2_dtype dtype, cudaStream_t s);

// ---- mixture of experts (moe.cu) ---------------------------------------------------
// Scores, choice and sorting of T tokens from router logits [T][E].
int moe_route(const float *logits, int T, const MoeRoute &r, cudaStream_t s);
// Routing by token id: row id of `table` [vocab][top] names the token's experts.
struct MoeTable {
    const int *table;
    MoeRoute r;            // r.pairs is not read
};
// Sorting of T tokens for `n` such layers at once (tables_dev: device memory).
int moe_route_tables(const MoeTable *tables_dev, int n, const uint32_t *ids, int vocab, int T, cudaStream_t s);

// ---- the stack ---------------------------------------------------------------------
struct Stack;
int stack_create(Stack **out, const ab2_model_config &cfg, const ab2_layer_spec *specs, ab2_dtype dtype, int max_tokens);
void stack_destroy(Stack *st);
int stack_set_linear(Stack *st, int layer, int which, const ab2_qweight *w);
int stack_set_norm(Stack *st, int layer, int which, const float *weight);
int stack_set_form(Stack *st, const ab2_stack_form &form);
int stack_set_loop_steps(Stack *st, const float *steps);
int stack_set_expert_table(Stack *st, int layer, const int *table);
int stack_runs(const Stack *st);   // layers run in a pass, each with a cache layer of its own
int stack_finalize(Stack *st);
int stack_check_cache(const Stack *st, const ab2_kv *kv, int S);
int stack_forward(Stack *st, ab2_kv *kv, const uint32_t *ids, int S, int row0, int nrows, int logits_mode, float *logits,
                  uint32_t *argmax_out, int len_hint, cudaStream_t s);

}  // namespace ab2
