// Layer stacks: a decoder whose layers are listed one by one, each with its mixer and feed-forward,
// over an f32 residual stream with the norms on the sublayers' outputs:
//   x = norm(embedding);   x += norm1(mixer(x));   x += norm2(ffn(x));   logits = head . norm(x)
// The handle, the step functions, the cache and graph replay are those of model.cu; this file holds
// the layers' weights, the workspace and the launches of a pass.
#include <algorithm>
#include <cmath>
#include <cstring>
#include <map>

#include "ops.cuh"
#include "stack.cuh"

using namespace ab2;

namespace ab2 {
int device_status_word(int **out);

struct StackLayer {
    ab2_layer_spec spec;
    std::vector<float> decay;
    const ab2_qweight *in, *out, *gate, *up, *down, *router;  // borrowed
    float *norm1, *norm2, *mix_norm;                            // owned, device
    const float *cos_t, *sin_t;                                 // attention; owned by Stack::tables
    float *decay_pow;                                           // lightning; owned
    int v_mode;                                                 // attention: WindowPrepArgs::v_mode
    int proj_width() const {
        return spec.mixer == AB2_MIX_LIGHTNING ? 2 * spec.heads * (spec.dim + spec.vdim)
                                               : (spec.heads + spec.kv_heads) * spec.dim + spec.kv_heads * spec.vdim;
    }
};

struct Stack {
    ab2_model_config cfg;
    ab2_dtype dtype;
    int max_tokens;
    std::vector<StackLayer> layers;
    const ab2_qweight *embedding, *lm_head;
    float *embed_norm, *final_norm;
    std::map<std::pair<int, double>, std::pair<float *, float *>> tables;  // (dims, base) -> cos, sin
    // workspace, sized for max_tokens
    float *x, *mix32, *parts, *router_z;
    void *xb, *proj, *mixed, *act, *gathered, *v_first, *head_in;
    int *route_int;
    float *route_score, *logits_scratch, *seg_states;
    bool ready;
};

#define STEP(expr)                     \
    do {                               \
        int _rc = (expr);              \
        if (_rc != AB2_OK) return _rc; \
    } while (0)

static int check_spec(const ab2_layer_spec &sp, int i) {
    AB2_REQUIRE(sp.mixer == AB2_MIX_ATTENTION || sp.mixer == AB2_MIX_LIGHTNING, AB2_ERR_BAD_ARG, "layer %d: unknown mixer %d", i, sp.mixer);
    AB2_REQUIRE(sp.heads > 0 && sp.dim > 0 && sp.vdim > 0, AB2_ERR_BAD_SHAPE, "layer %d: mixer sizes must be positive", i);
    AB2_REQUIRE(sp.dim <= 256 && sp.vdim <= 256, AB2_ERR_UNSUPPORTED, "layer %d: head sizes up to 256 are served, got %d and %d", i, sp.dim, sp.vdim);
    if (sp.mixer == AB2_MIX_ATTENTION) {
        AB2_REQUIRE(sp.kv_heads > 0 && sp.heads % sp.kv_heads == 0, AB2_ERR_BAD_SHAPE, "layer %d: %d query heads are not a multiple of %d KV heads", i, sp.heads, sp.kv_heads);
        AB2_REQUIRE(sp.window >= 0, AB2_ERR_BAD_SHAPE, "layer %d: negative window", i);
        AB2_REQUIRE(sp.rot_dims >= 0 && sp.rot_dims <= sp.dim && sp.rot_dims % 2 == 0, AB2_ERR_BAD_SHAPE, "layer %d: %d rotated dimensions of %d", i, sp.rot_dims, sp.dim);
    } else {
        AB2_REQUIRE(sp.decay != nullptr, AB2_ERR_BAD_ARG, "layer %d: no decays", i);
    }
    AB2_REQUIRE(sp.ffn == AB2_FFN_NONE || sp.ffn == AB2_FFN_MOE, AB2_ERR_BAD_ARG, "layer %d: unknown feed-forward %d", i, sp.ffn);
    if (sp.ffn == AB2_FFN_MOE)
        AB2_REQUIRE(sp.experts > 0 && sp.experts <= 1024 && sp.top > 0 && sp.top <= sp.experts && sp.ff > 0, AB2_ERR_BAD_SHAPE,
                    "layer %d: %d of %d experts of width %d", i, sp.top, sp.experts, sp.ff);
    return AB2_OK;
}

int stack_create(Stack **out, const ab2_model_config &cfg, const ab2_layer_spec *specs, ab2_dtype dtype, int max_tokens) {
    AB2_REQUIRE(cfg.n_layers > 0 && cfg.d_model > 0 && cfg.vocab > 0 && cfg.max_seq > 0, AB2_ERR_BAD_SHAPE, "model dimensions must be positive");
    AB2_REQUIRE(dtype == AB2_F32 || dtype == AB2_BF16, AB2_ERR_BAD_DTYPE, "a layer stack computes in f32 or bf16, got %d", (int)dtype);
    AB2_REQUIRE(max_tokens > 0 && max_tokens <= 65535, AB2_ERR_BAD_SHAPE, "max_tokens must be in 1..65535, got %d", max_tokens);
    int first_mix = -1;
    for (int i = 0; i < cfg.n_layers; ++i) {
        STEP(check_spec(specs[i], i));
        if (specs[i].mixer != AB2_MIX_ATTENTION || !specs[i].v_mix) continue;
        if (first_mix < 0) first_mix = i;
        AB2_REQUIRE(specs[i].kv_heads == specs[first_mix].kv_heads && specs[i].vdim == specs[first_mix].vdim, AB2_ERR_BAD_SHAPE,
                    "layers %d and %d mix values of different sizes", first_mix, i);
    }
    Stack *st = new Stack();
    st->cfg = cfg; st->dtype = dtype; st->max_tokens = max_tokens;
    st->layers.resize(cfg.n_layers);
    for (int i = 0; i < cfg.n_layers; ++i) {
        StackLayer &L = st->layers[i];
        L = StackLayer();
        L.spec = specs[i];
        if (L.spec.mixer == AB2_MIX_LIGHTNING) L.decay.assign(specs[i].decay, specs[i].decay + specs[i].heads);
        L.spec.decay = nullptr;
        if (L.spec.mixer == AB2_MIX_ATTENTION && L.spec.v_mix) L.v_mode = i == first_mix ? 1 : 2;
    }
    *out = st;
    return AB2_OK;
}

static void free_workspace(Stack *st) {
    void **all[] = {(void **)&st->x, (void **)&st->mix32, (void **)&st->parts, (void **)&st->router_z, &st->xb, &st->proj, &st->mixed,
                    &st->act, &st->gathered, &st->v_first, &st->head_in, (void **)&st->route_int, (void **)&st->route_score,
                    (void **)&st->logits_scratch, (void **)&st->seg_states};
    for (void **p : all) { cudaFree(*p); *p = nullptr; }
}

void stack_destroy(Stack *st) {
    if (!st) return;
    free_workspace(st);
    for (auto &L : st->layers) { cudaFree(L.norm1); cudaFree(L.norm2); cudaFree(L.mix_norm); cudaFree(L.decay_pow); }
    for (auto &t : st->tables) { cudaFree(t.second.first); cudaFree(t.second.second); }
    cudaFree(st->embed_norm); cudaFree(st->final_norm);
    delete st;
}

int stack_set_linear(Stack *st, int layer, int which, const ab2_qweight *w) {
    const int d = st->cfg.d_model;
    int N, K = d;
    const ab2_qweight **slot;
    if (layer < 0) {
        AB2_REQUIRE(which == 0 || which == 1, AB2_ERR_BAD_ARG, "model-level weight index must be 0 (embedding) or 1 (lm_head)");
        slot = which == 0 ? &st->embedding : &st->lm_head;
        N = st->cfg.vocab;
    } else {
        AB2_REQUIRE(layer < st->cfg.n_layers, AB2_ERR_BAD_ARG, "layer %d out of range", layer);
        StackLayer &L = st->layers[layer];
        AB2_REQUIRE(which < 4 || L.spec.ffn == AB2_FFN_MOE, AB2_ERR_BAD_ARG, "layer %d has no feed-forward", layer);
        switch (which) {
        case 0: slot = &L.in; N = L.proj_width(); break;
        case 3: slot = &L.out; N = d; K = L.spec.heads * L.spec.vdim; break;
        case 4: slot = &L.gate; N = L.spec.experts * L.spec.ff; break;
        case 5: slot = &L.up; N = L.spec.experts * L.spec.ff; break;
        case 6: slot = &L.down; N = L.spec.experts * d; K = L.spec.ff; break;
        case 7: slot = &L.router; N = L.spec.experts; break;
        default: return fail(AB2_ERR_BAD_ARG, "a stack layer has no weight %d", which);
        }
    }
    AB2_REQUIRE(w->fmt == FMT_BF16, AB2_ERR_UNSUPPORTED, "a layer stack takes dense bf16 weights, got format %d", w->fmt);
    AB2_REQUIRE(w->N == N && w->K == K, AB2_ERR_BAD_SHAPE, "weight is [%d,%d], expected [%d,%d]", w->N, w->K, N, K);
    *slot = w;
    st->ready = false;
    return AB2_OK;
}

int stack_set_norm(Stack *st, int layer, int which, const float *weight) {
    float **slot;
    size_t n = st->cfg.d_model;
    if (layer < 0) {
        AB2_REQUIRE(which == 0 || which == 1, AB2_ERR_BAD_ARG, "model-level norm index must be 0 (final) or 1 (embedding)");
        slot = which == 0 ? &st->final_norm : &st->embed_norm;
    } else {
        AB2_REQUIRE(layer < st->cfg.n_layers && which >= 0 && which <= 2, AB2_ERR_BAD_ARG, "layer %d / norm %d out of range", layer, which);
        StackLayer &L = st->layers[layer];
        AB2_REQUIRE(which != 2 || L.spec.mixer == AB2_MIX_LIGHTNING, AB2_ERR_BAD_ARG, "layer %d has no norm inside its mixer", layer);
        slot = which == 0 ? &L.norm1 : which == 1 ? &L.norm2 : &L.mix_norm;
        if (which == 2) n = (size_t)L.spec.heads * L.spec.vdim;
    }
    if (!*slot) AB2_CUDA(cudaMalloc((void **)slot, n * 4));
    AB2_CUDA(cudaMemcpy(*slot, weight, n * 4, cudaMemcpyDefault));
    return AB2_OK;
}

// cos / sin of position * base^(-2i / dims), the angle in f64 and rounded once.
static int rotation_tables(Stack *st, int dims, double base, const float **c, const float **s) {
    auto &t = st->tables[{dims, base}];
    if (!t.first) {
        const int half = dims / 2, n = st->cfg.max_seq;
        std::vector<float> cv((size_t)n * half), sv((size_t)n * half);
        for (int i = 0; i < half; ++i) {
            const double f = std::pow(base, -2.0 * i / dims);
            for (int p = 0; p < n; ++p) {
                cv[(size_t)p * half + i] = (float)std::cos(p * f);
                sv[(size_t)p * half + i] = (float)std::sin(p * f);
            }
        }
        AB2_CUDA(cudaMalloc((void **)&t.first, cv.size() * 4));
        AB2_CUDA(cudaMalloc((void **)&t.second, sv.size() * 4));
        AB2_CUDA(cudaMemcpy(t.first, cv.data(), cv.size() * 4, cudaMemcpyHostToDevice));
        AB2_CUDA(cudaMemcpy(t.second, sv.data(), sv.size() * 4, cudaMemcpyHostToDevice));
    }
    *c = t.first; *s = t.second;
    return AB2_OK;
}

int stack_finalize(Stack *st) {
    const size_t T = st->max_tokens, esz = dtype_size(st->dtype), d = st->cfg.d_model;
    AB2_REQUIRE(st->embedding && st->embed_norm && st->final_norm, AB2_ERR_BAD_ARG, "embedding or a model-level norm not set");
    if (!st->lm_head) {
        AB2_REQUIRE(st->cfg.tied, AB2_ERR_BAD_ARG, "lm_head not set and embeddings are not tied");
        st->lm_head = st->embedding;
    }
    size_t proj = 0, mixed = 0, mix32 = 0, parts = 1, act = 0, gathered = 0, z = 0, vf = 0, pairs = 0, experts = 0, state = 0;
    for (int i = 0; i < st->cfg.n_layers; ++i) {
        StackLayer &L = st->layers[i];
        const ab2_layer_spec &sp = L.spec;
        AB2_REQUIRE(L.in && L.out && L.norm1, AB2_ERR_BAD_ARG, "layer %d: a weight or norm of the mixer is not set", i);
        const size_t hv = (size_t)sp.heads * sp.vdim;
        proj = std::max(proj, (size_t)L.proj_width());
        mixed = std::max(mixed, hv);
        if (sp.mixer == AB2_MIX_LIGHTNING) {
            AB2_REQUIRE(L.mix_norm != nullptr, AB2_ERR_BAD_ARG, "layer %d: the mixer's norm is not set", i);
            mix32 = std::max(mix32, hv);
            state = std::max(state, hv * sp.dim);
            std::vector<float> pw((size_t)sp.heads * (LIGHTNING_CHUNK + 1));
            for (int h = 0; h < sp.heads; ++h)
                for (int n = 0; n <= LIGHTNING_CHUNK; ++n)
                    pw[(size_t)h * (LIGHTNING_CHUNK + 1) + n] = (float)std::pow((double)L.decay[h], n);
            if (!L.decay_pow) AB2_CUDA(cudaMalloc((void **)&L.decay_pow, pw.size() * 4));
            AB2_CUDA(cudaMemcpy(L.decay_pow, pw.data(), pw.size() * 4, cudaMemcpyHostToDevice));
        } else {
            if (sp.rot_dims > 0) STEP(rotation_tables(st, sp.rot_dims, sp.rot_base, &L.cos_t, &L.sin_t));
            if (sp.v_mix) vf = std::max(vf, (size_t)sp.kv_heads * sp.vdim);
        }
        if (sp.ffn == AB2_FFN_MOE) {
            AB2_REQUIRE(L.gate && L.up && L.down && L.router && L.norm2, AB2_ERR_BAD_ARG, "layer %d: a weight or norm of the feed-forward is not set", i);
            parts = std::max(parts, (size_t)sp.top);
            act = std::max(act, (size_t)sp.top * sp.ff);
            gathered = std::max(gathered, (size_t)sp.top * d);
            z = std::max(z, (size_t)sp.experts);
            pairs = std::max(pairs, (size_t)sp.top);
            experts = std::max(experts, (size_t)sp.experts);
        }
    }
    if (!st->x) {
        const bool b16 = st->dtype != AB2_F32;
        struct { void **p; size_t bytes; } all[] = {
            {(void **)&st->x, T * d * 4}, {&st->xb, b16 ? T * d * esz : 0}, {&st->proj, T * proj * esz}, {&st->mixed, T * mixed * esz},
            {(void **)&st->mix32, T * mix32 * 4}, {(void **)&st->parts, T * parts * d * 4}, {&st->act, T * act * esz},
            {&st->gathered, b16 ? T * gathered * esz : 0}, {(void **)&st->router_z, T * z * 4}, {&st->v_first, T * vf * esz},
            {&st->head_in, T * d * esz}, {(void **)&st->route_int, (T * pairs * 2 + 2 * (experts + 1)) * 4},
            {(void **)&st->route_score, T * pairs * 4}, {(void **)&st->logits_scratch, T * st->cfg.vocab * 4}, 
            {(void **)&st->seg_states, b16 ? LIGHTNING_MAX_SEGMENTS * state * 4 : 0}};
        for (auto &a : all) {
            if (a.bytes == 0) continue;
            cudaError_t e = cudaMalloc(a.p, a.bytes);
            if (e != cudaSuccess) {
                free_workspace(st);
                return fail(AB2_ERR_CUDA, "workspace allocation of %zu bytes failed: %s", a.bytes, cudaGetErrorString(e));
            }
        }
    }
    int *status_word = nullptr;  // allocate the device status word outside any capture
    STEP(device_status_word(&status_word));
    st->ready = true;
    return AB2_OK;
}

int stack_check_cache(const Stack *st, const ab2_kv *kv, int S) {
    AB2_REQUIRE(kv->layers != nullptr, AB2_ERR_BAD_SHAPE, "a layer stack needs a cache of ab2_kv_create_stack");
    AB2_REQUIRE(kv->dtype == (st->dtype == AB2_F32 ? AB2_KV_F32 : AB2_KV_BF16), AB2_ERR_BAD_DTYPE, "the cache's type differs from the model's");
    for (int i = 0; i < kv->L; ++i) {
        const KvLayer &l = kv->layers[i];
        const ab2_layer_spec &sp = st->layers[i].spec;
        const bool rec = sp.mixer == AB2_MIX_LIGHTNING;
        AB2_REQUIRE(l.recurrent == rec && l.kvh == (rec ? sp.heads : sp.kv_heads) && l.kd == sp.dim && l.vd == sp.vdim &&
                        (rec || l.window == (sp.window > 0 ? std::min(sp.window, kv->cap) : kv->cap)),
                    AB2_ERR_BAD_SHAPE, "cache layer %d does not match the model", i);
        AB2_REQUIRE(rec || l.cap == kv->cap || l.window - 1 + S <= l.cap, AB2_ERR_CAPACITY,
                    "a step of %d tokens exceeds the %d the cache was made for", S, l.cap - l.window + 1);
    }
    return AB2_OK;
}

static int attention_mixer(Stack *st, StackLayer &L, ab2_kv *kv, int layer, int S, int row0, int nrows, int max_len, cudaStream_t s) {
    const ab2_layer_spec &sp = L.spec;
    WindowPrepArgs p = {};
    p.kv = kv_layer_view(kv, layer);
    p.qkv = st->proj; p.stride = L.proj_width(); p.S = S; p.row0 = row0; p.H = sp.heads; p.G = sp.kv_heads; p.dim = sp.dim; p.vdim = sp.vdim;
    p.rot_dims = sp.rot_dims; p.qk_norm = sp.qk_norm; p.cos_t = L.cos_t; p.sin_t = L.sin_t; p.eps = st->cfg.rms_eps;
    p.v_first = st->v_first; p.v_mode = L.v_mode; p.lambda = sp.v_lambda;
    WindowAttnArgs a = {};
    a.prep = p; a.kv = p.kv; a.q = st->proj; a.q_stride = p.stride; a.out = st->mixed; a.S = S; a.row0 = row0; a.H = sp.heads;
    a.rep = sp.heads / sp.kv_heads; a.dim = sp.dim; a.vdim = sp.vdim; a.scale = sp.scale;
    return window_attention(kv, a, nrows, max_len, st->dtype, s);
}

static int lightning_mixer(Stack *st, StackLayer &L, ab2_kv *kv, int layer, int S, int row0, int nrows, cudaStream_t s) {
    const ab2_layer_spec &sp = L.spec;
    LightningArgs a = {};
    a.kv = kv_layer_view(kv, layer);
    a.qkv = st->proj; a.stride = L.proj_width(); a.out = st->mix32; a.S = S; a.row0 = row0; a.H = sp.heads; a.dim = sp.dim; a.vdim = sp.vdim;
    a.decay_pow = L.decay_pow; a.scratch = st->seg_states;
    ResidualNormArgs n = {};
    n.w = L.mix_norm; n.eps = st->cfg.rms_eps; n.d = sp.heads * sp.vdim; n.parts = st->mix32; n.out = st->mixed;
    n.gate = (const char *)st->proj + (size_t)sp.heads * (2 * sp.dim + sp.vdim) * dtype_size(st->dtype);
    n.gate_stride = a.stride;
    STEP(lightning_attention(a, nrows, st->dtype, s));
    return launch_residual_norm(n, RN_GATED, nrows * S, st->dtype, s);
}

// Scratch of a mixture of experts.
struct MoeScratch {
    float *router_z;       // [T][experts]
    int *route_int;        // 2 T top + 2 (experts + 1)
    float *route_score;    // [T top]
    void *act, *gathered;  // [T top][ff], [T top][width] in the activation type
};

// parts[t * top + slot] = W_down glu(s W_gate x_t, s W_up x_t) of the token's slot-th expert, f32
static int moe_experts(const ab2_layer_spec &sp, const ab2_qweight *router, const ab2_qweight *gate, const ab2_qweight *up,
                       const ab2_qweight *down, const void *in, int T, ab2_dtype dtype, const MoeScratch &w, float *parts, cudaStream_t s) {
    MoeRoute r = {};
    r.E = sp.experts; r.top = sp.top; r.pairs = T * sp.top;
    r.perm = w.route_int; r.expert = r.perm + r.pairs; r.offset = r.expert + r.pairs; r.active = r.offset + sp.experts + 1;
    r.score = w.route_score;
    STEP(linear_bf16(router, in, T, dtype, w.router_z, LIN_F32, 0, s));
    STEP(moe_route(w.router_z, T, r, s));
    STEP(linear_moe_glu(gate, up, in, dtype, w.act, sp.limit, r, w.gathered, s));
    return linear_moe_down(down, w.act, dtype, parts, r, s);
}

static int moe_ffn(Stack *st, StackLayer &L, const void *in, int T, cudaStream_t s) {
    const MoeScratch w = {st->router_z, st->route_int, st->route_score, st->act, st->gathered};
    return moe_experts(L.spec, L.router, L.gate, L.up, L.down, in, T, st->dtype, w, st->parts, s);
}

int stack_forward(Stack *st, ab2_kv *kv, const uint32_t *ids, int S, int row0, int nrows, int logits_mode, float *logits,
                  uint32_t *argmax_out, int len_hint, cudaStream_t s) {
    const int T = nrows * S, d = st->cfg.d_model;
    int max_len = len_hint;
    if (max_len <= 0)
        for (int i = 0; i < nrows; ++i) max_len = std::max(max_len, kv->lens_host[kv_row_host(kv, row0, i)] + S);
    const void *in = st->dtype == AB2_F32 ? (const void *)st->x : st->xb;  // what the sublayers read
    ResidualNormArgs n = {};
    n.eps = st->cfg.rms_eps; n.d = d; n.x = st->x; n.out = st->xb;
    n.w = st->embed_norm; n.table = (const __nv_bfloat16 *)st->embedding->codes; n.ids = ids; n.vocab = st->cfg.vocab;
    STEP(launch_residual_norm(n, RN_EMBED, T, st->dtype, s));
    n.parts = st->parts;
    for (int l = 0; l < st->cfg.n_layers; ++l) {
        StackLayer &L = st->layers[l];
        const ab2_layer_spec &sp = L.spec;
        if (sp.mixer == AB2_MIX_LIGHTNING) {
            STEP(linear_bf16(L.in, in, T, st->dtype, st->proj, LIN_ACT, sp.heads * (2 * sp.dim + sp.vdim), s));
            STEP(lightning_mixer(st, L, kv, l, S, row0, nrows, s));
        } else {
            STEP(linear_bf16(L.in, in, T, st->dtype, st->proj, LIN_STORE, 0, s));
            STEP(attention_mixer(st, L, kv, l, S, row0, nrows, max_len, s));
        }
        STEP(linear_bf16(L.out, st->mixed, T, st->dtype, st->parts, LIN_F32, 0, s));
        n.w = L.norm1; n.nparts = 1;
        STEP(launch_residual_norm(n, RN_ADD, T, st->dtype, s));
        if (sp.ffn == AB2_FFN_NONE) continue;
        STEP(moe_ffn(st, L, in, T, s));
        n.w = L.norm2; n.nparts = sp.top;
        STEP(launch_residual_norm(n, RN_ADD, T, st->dtype, s));
    }
    if (logits_mode == 0 && argmax_out == nullptr) return AB2_OK;
    const bool last = logits_mode != 2;
    const int rows = last ? nrows : T;
    AB2_REQUIRE(!argmax_out || last || S == 1, AB2_ERR_UNSUPPORTED, "argmax with all-token logits needs S == 1");
    n.w = st->final_norm; n.step = last ? S : 1; n.out = st->head_in;
    STEP(launch_residual_norm(n, RN_FINAL, rows, st->dtype, s));
    float *lg = logits ? logits : st->logits_scratch;
    STEP(linear_bf16(st->lm_head, st->head_in, rows, st->dtype, lg, LIN_F32, 0, s));
    if (argmax_out) STEP(launch_argmax(lg, nrows, st->cfg.vocab, AB2_F32, argmax_out, s));
    return AB2_OK;
}

}  // namespace ab2

// ---- the mechanisms as operators of their own ---------------------------------------

static int check_mixer_call(const ab2_kv *kv, int layer, const ab2_layer_spec *spec, int mixer, const void *qkv, const void *out, int S,
                            int row0, int nrows, ab2_dtype dtype) {
    AB2_REQUIRE(kv && spec && qkv && out, AB2_ERR_BAD_ARG, "null argument");
    AB2_REQUIRE(kv->layers && layer >= 0 && layer < kv->L, AB2_ERR_BAD_SHAPE, "layer %d of a stack cache expected", layer);
    AB2_REQUIRE(spec->mixer == mixer, AB2_ERR_BAD_ARG, "the spec names another mixer");
    if (mixer == AB2_MIX_ATTENTION) STEP(check_spec(*spec, layer));
    const KvLayer &l = kv->layers[layer];
    const bool rec = mixer == AB2_MIX_LIGHTNING;
    AB2_REQUIRE(l.recurrent == rec && l.kvh == (rec ? spec->heads : spec->kv_heads) && l.kd == spec->dim && l.vd == spec->vdim,
                AB2_ERR_BAD_SHAPE, "cache layer %d does not match the spec", layer);
    AB2_REQUIRE(dtype == AB2_F32 || dtype == AB2_BF16, AB2_ERR_BAD_DTYPE, "unsupported dtype %d", (int)dtype);
    AB2_REQUIRE(kv->dtype == (dtype == AB2_F32 ? AB2_KV_F32 : AB2_KV_BF16), AB2_ERR_BAD_DTYPE, "the cache's type differs from the activations'");
    AB2_REQUIRE(S > 0 && nrows > 0 && row0 >= 0 && row0 + nrows <= kv->B && (long long)nrows * S <= 65535, AB2_ERR_BAD_SHAPE,
                "rows %d..%d of %d tokens do not fit", row0, row0 + nrows, S);
    AB2_REQUIRE(rec || l.cap == kv->cap || l.window - 1 + S <= l.cap, AB2_ERR_CAPACITY, "a step of %d tokens exceeds what the cache was made for", S);
    for (int i = 0; i < nrows; ++i)
        AB2_REQUIRE(kv->lens_host[row0 + i] + S <= kv->cap, AB2_ERR_CAPACITY, "KV cache length %d exceeds capacity %d", kv->lens_host[row0 + i] + S, kv->cap);
    return AB2_OK;
}

AB2_API int ab2_window_attention(ab2_kv *kv, int layer, const ab2_layer_spec *spec, void *qkv_dev, void *v_first_dev, int v_mode,
                                 const float *cos_dev, const float *sin_dev, float eps, void *out_dev, int S, int row0, int nrows,
                                 ab2_dtype dtype, ab2_stream stream) {
    STEP(check_mixer_call(kv, layer, spec, AB2_MIX_ATTENTION, qkv_dev, out_dev, S, row0, nrows, dtype));
    AB2_REQUIRE(spec->rot_dims == 0 || (cos_dev && sin_dev), AB2_ERR_BAD_ARG, "null rotation tables");
    AB2_REQUIRE(v_mode >= 0 && v_mode <= 2 && (v_mode == 0 || v_first_dev), AB2_ERR_BAD_ARG, "value mixing %d needs the first values", v_mode);
    WindowPrepArgs p = {};
    p.kv = kv_layer_view(kv, layer);
    p.qkv = qkv_dev; p.stride = (long long)(spec->heads + spec->kv_heads) * spec->dim + (long long)spec->kv_heads * spec->vdim;
    p.S = S; p.row0 = row0; p.H = spec->heads; p.G = spec->kv_heads; p.dim = spec->dim; p.vdim = spec->vdim;
    p.rot_dims = spec->rot_dims; p.qk_norm = spec->qk_norm; p.cos_t = cos_dev; p.sin_t = sin_dev; p.eps = eps;
    p.v_first = v_first_dev; p.v_mode = v_mode; p.lambda = spec->v_lambda;
    WindowAttnArgs a = {};
    a.prep = p; a.kv = p.kv; a.q = qkv_dev; a.q_stride = p.stride; a.out = out_dev; a.S = S; a.row0 = row0; a.H = spec->heads;
    a.rep = spec->heads / spec->kv_heads; a.dim = spec->dim; a.vdim = spec->vdim; a.scale = spec->scale;
    int max_len = 0;
    for (int i = 0; i < nrows; ++i) max_len = std::max(max_len, kv->lens_host[row0 + i] + S);
    return window_attention(kv, a, nrows, max_len, dtype, (cudaStream_t)stream);
}

AB2_API int ab2_lightning_attention(ab2_kv *kv, int layer, const ab2_layer_spec *spec, const float *decay_pow_dev, const void *qkv_dev,
                                    long long stride, float *scratch_dev, float *out_dev, int S, int row0, int nrows, ab2_dtype dtype, ab2_stream stream) {
    STEP(check_mixer_call(kv, layer, spec, AB2_MIX_LIGHTNING, qkv_dev, out_dev, S, row0, nrows, dtype));
    AB2_REQUIRE(decay_pow_dev != nullptr, AB2_ERR_BAD_ARG, "null decay table");
    AB2_REQUIRE(stride >= (long long)spec->heads * (2 * spec->dim + spec->vdim), AB2_ERR_BAD_SHAPE, "row stride %lld is too short", stride);
    LightningArgs a = {};
    a.kv = kv_layer_view(kv, layer);
    a.qkv = qkv_dev; a.stride = stride; a.out = out_dev; a.S = S; a.row0 = row0; a.H = spec->heads; a.dim = spec->dim; a.vdim = spec->vdim;
    a.decay_pow = decay_pow_dev; a.scratch = scratch_dev;
    return lightning_attention(a, nrows, dtype, (cudaStream_t)stream);
}

static size_t up256(size_t n) { return (n + 255) / 256 * 256; }

AB2_API int ab2_moe_workspace(const ab2_layer_spec *spec, int width, int tokens, ab2_dtype dtype, size_t *bytes) {
    AB2_REQUIRE(spec && bytes, AB2_ERR_BAD_ARG, "null argument");
    AB2_REQUIRE(width > 0 && tokens > 0 && spec->experts > 0 && spec->top > 0 && spec->ff > 0, AB2_ERR_BAD_SHAPE, "sizes must be positive");
    const size_t P = (size_t)tokens * spec->top, esz = dtype_size(dtype);
    *bytes = up256((size_t)tokens * spec->experts * 4) + up256((2 * P + 2 * (spec->experts + 1)) * 4) + up256(P * 4) + up256(P * spec->ff * esz) +
             up256(P * width * esz);
    return AB2_OK;
}

AB2_API int ab2_moe_forward(const ab2_layer_spec *spec, const ab2_qweight *router, const ab2_qweight *gate, const ab2_qweight *up,
                            const ab2_qweight *down, const void *x_dev, int tokens, ab2_dtype dtype, float *parts_dev, void *workspace_dev,
                            ab2_stream stream) {
    AB2_REQUIRE(spec && router && gate && up && down && x_dev && parts_dev && workspace_dev, AB2_ERR_BAD_ARG, "null argument");
    AB2_REQUIRE(tokens > 0 && spec->experts > 0 && spec->experts <= 1024 && spec->top > 0 && spec->top <= spec->experts && spec->ff > 0,
                AB2_ERR_BAD_SHAPE, "%d of %d experts of width %d over %d tokens", spec->top, spec->experts, spec->ff, tokens);
    AB2_REQUIRE(dtype == AB2_F32 || dtype == AB2_BF16, AB2_ERR_BAD_DTYPE, "unsupported dtype %d", (int)dtype);
    const int E = spec->experts, d = router->K;
    for (const ab2_qweight *w : {router, gate, up, down}) AB2_REQUIRE(w->fmt == FMT_BF16, AB2_ERR_UNSUPPORTED, "experts are dense bf16 weights");
    AB2_REQUIRE(router->N == E && gate->N == E * spec->ff && up->N == gate->N && gate->K == d && up->K == d && down->N == E * d && down->K == spec->ff,
                AB2_ERR_BAD_SHAPE, "the experts' weights do not match the spec");
    const size_t P = (size_t)tokens * spec->top, esz = dtype_size(dtype);
    char *p = (char *)workspace_dev;
    MoeScratch w;
    w.router_z = (float *)p; p += up256((size_t)tokens * E * 4);
    w.route_int = (int *)p; p += up256((2 * P + 2 * (E + 1)) * 4);
    w.route_score = (float *)p; p += up256(P * 4);
    w.act = p; p += up256(P * spec->ff * esz);
    w.gathered = p;
    return moe_experts(*spec, router, gate, up, down, x_dev, tokens, dtype, w, parts_dev, (cudaStream_t)stream);
}
