// Layer stacks: a decoder whose layers are listed one by one, each with its mixer and feed-forward,
// over an f32 residual stream with norms on the sublayers' outputs:
//   x = norm(embedding);   x += norm1(mixer(x));   x += norm2(ffn(x));   logits = head . norm(x)
// As ab2_stack_form says, the embedding stays as it is, sublayers read a norm of x, some layers run
// several times in a row (each run with a cache layer of its own), and the logits are capped.
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
    const ab2_qweight *ukv, *shared_gate, *shared_up, *shared_down;
    float *norm1, *norm2, *mix_norm, *pre1, *pre2;              // owned, device
    const float *cos_t, *sin_t;                                 // attention; owned by Stack::tables
    __nv_bfloat16 *absorb;                                      // latent: ab2::latent_absorb_weights of ukv; owned
    int *table, *route_int;                                     // experts by token id, and their routing; owned
    float *decay_pow;                                           // lightning; owned
    int v_mode;                                                 // attention: WindowPrepArgs::v_mode
    int proj_width() const {
        if (spec.mixer == AB2_MIX_LATENT)  // rows of 16 bytes
            return (spec.heads * (spec.dim + spec.rot_dims) + spec.kv_rank + spec.rot_dims + (spec.head_gate ? spec.heads : 0) + 7) / 8 * 8;
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
    ab2_stack_form form;
    float *loop_steps;            // [loop_times][d_model], owned
    struct Run { int layer, pass; };  // pass: of the loop, at its first layer; else -1
    std::vector<Run> runs;
    MoeTable *route_tables;       // of the layers with experts by token id, device
    int n_route_tables;
    std::map<std::pair<int, double>, std::pair<float *, float *>> tables;  // (dims, base) -> cos, sin
    // workspace, sized for max_tokens
    float *x, *x0, *mix32, *parts, *router_z, *shared_out;
    void *shared_act, *z, *latent_work;
    size_t latent_bytes;
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
    AB2_REQUIRE(sp.mixer == AB2_MIX_ATTENTION || sp.mixer == AB2_MIX_LIGHTNING || sp.mixer == AB2_MIX_LATENT, AB2_ERR_BAD_ARG,
                "layer %d: unknown mixer %d", i, sp.mixer);
    AB2_REQUIRE(sp.heads > 0 && sp.dim > 0 && sp.vdim > 0, AB2_ERR_BAD_SHAPE, "layer %d: mixer sizes must be positive", i);
    AB2_REQUIRE(sp.dim <= 256 && sp.vdim <= 256, AB2_ERR_UNSUPPORTED, "layer %d: head sizes up to 256 are served, got %d and %d", i, sp.dim, sp.vdim);
    if (sp.mixer == AB2_MIX_ATTENTION) {
        AB2_REQUIRE(sp.kv_heads > 0 && sp.heads % sp.kv_heads == 0, AB2_ERR_BAD_SHAPE, "layer %d: %d query heads are not a multiple of %d KV heads", i, sp.heads, sp.kv_heads);
        AB2_REQUIRE(sp.window >= 0, AB2_ERR_BAD_SHAPE, "layer %d: negative window", i);
        AB2_REQUIRE(sp.rot_dims >= 0 && sp.rot_dims <= sp.dim && sp.rot_dims % 2 == 0, AB2_ERR_BAD_SHAPE, "layer %d: %d rotated dimensions of %d", i, sp.rot_dims, sp.dim);
    } else if (sp.mixer == AB2_MIX_LATENT) {
        AB2_REQUIRE(sp.kv_rank > 0 && sp.rot_dims >= 0 && sp.rot_dims % 2 == 0, AB2_ERR_BAD_SHAPE, "layer %d: latent of %d and %d rotated dimensions", i, sp.kv_rank, sp.rot_dims);
        AB2_REQUIRE(sp.kv_rank <= 1024 && sp.rot_dims <= 256, AB2_ERR_UNSUPPORTED, "layer %d: latents up to 1024 with 256 rotated dimensions are served, got %d and %d", i, sp.kv_rank, sp.rot_dims);
    } else {
        AB2_REQUIRE(sp.decay != nullptr, AB2_ERR_BAD_ARG, "layer %d: no decays", i);
    }
    AB2_REQUIRE(sp.ffn == AB2_FFN_NONE || sp.ffn == AB2_FFN_MOE || sp.ffn == AB2_FFN_POLY, AB2_ERR_BAD_ARG, "layer %d: unknown feed-forward %d", i, sp.ffn);
    AB2_REQUIRE(sp.ffn != AB2_FFN_POLY || sp.ff > 0, AB2_ERR_BAD_SHAPE, "layer %d: feed-forward of width %d", i, sp.ff);
    if (sp.ffn == AB2_FFN_MOE) {
        AB2_REQUIRE((sp.glu == AB2_GLU_CLAMPED || sp.glu == AB2_GLU_SILU) && (sp.routing == AB2_ROUTE_SIGMOID || sp.routing == AB2_ROUTE_TABLE) && sp.shared_ff >= 0,
                    AB2_ERR_BAD_ARG, "layer %d: unknown gated unit %d or routing %d", i, sp.glu, sp.routing);
        AB2_REQUIRE(sp.experts > 0 && sp.experts <= 1024 && sp.top > 0 && sp.top <= sp.experts && sp.ff > 0, AB2_ERR_BAD_SHAPE,
                    "layer %d: %d of %d experts of width %d", i, sp.top, sp.experts, sp.ff);
    }
    return AB2_OK;
}

static void list_runs(Stack *st) {
    const ab2_stack_form &f = st->form;
    const int loops = f.loop_times, start = loops ? f.loop_start : 0, stop = loops ? f.loop_stop : 0;
    st->runs.clear();
    for (int i = 0; i < start; ++i) st->runs.push_back({i, -1});
    for (int t = 0; t < loops; ++t)
        for (int i = start; i < stop; ++i) st->runs.push_back({i, i == start ? t : -1});
    for (int i = stop; i < st->cfg.n_layers; ++i) st->runs.push_back({i, -1});
}

int stack_runs(const Stack *st) { return (int)st->runs.size(); }

int stack_set_form(Stack *st, const ab2_stack_form &f) {
    AB2_REQUIRE(f.loop_times >= 0 && f.loop_times <= 1024, AB2_ERR_BAD_SHAPE, "%d passes of a loop", f.loop_times);
    AB2_REQUIRE(f.loop_times == 0 || (f.loop_start >= 0 && f.loop_start < f.loop_stop && f.loop_stop <= st->cfg.n_layers), AB2_ERR_BAD_SHAPE,
                "a loop over layers %d .. %d of %d", f.loop_start, f.loop_stop, st->cfg.n_layers);
    AB2_REQUIRE(f.logit_softcap >= 0.f, AB2_ERR_BAD_ARG, "negative cap of the logits");
    for (int i = f.loop_start; i < f.loop_stop && f.loop_times > 1; ++i)
        AB2_REQUIRE(st->layers[i].v_mode == 0, AB2_ERR_UNSUPPORTED, "layer %d mixes its values with the first layer's: it cannot be looped over", i);
    st->form = f;
    list_runs(st);
    st->ready = false;
    return AB2_OK;
}

int stack_set_loop_steps(Stack *st, const float *steps) {
    const size_t n = (size_t)st->form.loop_times * st->cfg.d_model;
    AB2_REQUIRE(n > 0, AB2_ERR_BAD_ARG, "the stack has no loop");
    cudaFree(st->loop_steps);
    AB2_CUDA(cudaMalloc((void **)&st->loop_steps, n * 4));
    AB2_CUDA(cudaMemcpy(st->loop_steps, steps, n * 4, cudaMemcpyDefault));
    return AB2_OK;
}

int stack_set_expert_table(Stack *st, int layer, const int *table) {
    AB2_REQUIRE(layer >= 0 && layer < st->cfg.n_layers, AB2_ERR_BAD_ARG, "layer %d out of range", layer);
    StackLayer &L = st->layers[layer];
    AB2_REQUIRE(L.spec.ffn == AB2_FFN_MOE && L.spec.routing == AB2_ROUTE_TABLE, AB2_ERR_BAD_ARG, "layer %d does not choose experts by token id", layer);
    std::vector<int> host((size_t)st->cfg.vocab * L.spec.top);
    AB2_CUDA(cudaMemcpy(host.data(), table, host.size() * 4, cudaMemcpyDefault));
    for (size_t i = 0; i < host.size(); ++i) {
        AB2_REQUIRE(host[i] >= 0 && host[i] < L.spec.experts, AB2_ERR_BAD_ARG, "token %zu names expert %d of %d", i / L.spec.top, host[i], L.spec.experts);
        for (size_t j = i / L.spec.top * L.spec.top; j < i; ++j)
            AB2_REQUIRE(host[j] != host[i], AB2_ERR_BAD_ARG, "token %zu names expert %d twice", i / L.spec.top, host[i]);
    }
    if (!L.table) AB2_CUDA(cudaMalloc((void **)&L.table, host.size() * 4));
    AB2_CUDA(cudaMemcpy(L.table, host.data(), host.size() * 4, cudaMemcpyHostToDevice));
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
    st->form.embed_norm = 1;
    st->layers.resize(cfg.n_layers);
    for (int i = 0; i < cfg.n_layers; ++i) {
        StackLayer &L = st->layers[i];
        L = StackLayer();
        L.spec = specs[i];
        if (L.spec.mixer == AB2_MIX_LIGHTNING) L.decay.assign(specs[i].decay, specs[i].decay + specs[i].heads);
        L.spec.decay = nullptr;
        if (L.spec.mixer == AB2_MIX_ATTENTION && L.spec.v_mix) L.v_mode = i == first_mix ? 1 : 2;
    }
    list_runs(st);
    *out = st;
    return AB2_OK;
}

static void free_workspace(Stack *st) {
    void **all[] = {(void **)&st->x, (void **)&st->mix32, (void **)&st->parts, (void **)&st->router_z, &st->xb, &st->proj, &st->mixed,
                    &st->act, &st->gathered, &st->v_first, &st->head_in, (void **)&st->route_int, (void **)&st->route_score,
                    (void **)&st->logits_scratch, (void **)&st->seg_states, (void **)&st->x0, (void **)&st->shared_out, &st->shared_act,
                    &st->z, &st->latent_work, (void **)&st->route_tables};
    for (auto &L : st->layers) { cudaFree(L.route_int); L.route_int = nullptr; }
    for (void **p : all) { cudaFree(*p); *p = nullptr; }
}

void stack_destroy(Stack *st) {
    if (!st) return;
    free_workspace(st);
    for (auto &L : st->layers) { cudaFree(L.norm1); cudaFree(L.norm2); cudaFree(L.mix_norm); cudaFree(L.decay_pow); cudaFree(L.pre1); cudaFree(L.pre2); cudaFree(L.absorb); cudaFree(L.table); }
    for (auto &t : st->tables) { cudaFree(t.second.first); cudaFree(t.second.second); }
    cudaFree(st->embed_norm); cudaFree(st->final_norm); cudaFree(st->loop_steps);
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
        const bool moe = L.spec.ffn == AB2_FFN_MOE;
        AB2_REQUIRE(which < 4 || moe || (L.spec.ffn == AB2_FFN_POLY && (which == 5 || which == 6)), AB2_ERR_BAD_ARG, "layer %d has no weight %d", layer, which);
        AB2_REQUIRE(which != 1 || L.spec.mixer == AB2_MIX_LATENT, AB2_ERR_BAD_ARG, "layer %d has no up projection of a latent", layer);
        AB2_REQUIRE(which < 8 || L.spec.shared_ff > 0, AB2_ERR_BAD_ARG, "layer %d has no shared expert", layer);
        const int E = moe ? L.spec.experts : 1;
        switch (which) {
        case 1: slot = &L.ukv; N = L.spec.heads * (L.spec.dim + L.spec.vdim); K = L.spec.kv_rank; break;
        case 8: slot = &L.shared_gate; N = L.spec.shared_ff; break;
        case 9: slot = &L.shared_up; N = L.spec.shared_ff; break;
        case 10: slot = &L.shared_down; N = d; K = L.spec.shared_ff; break;
        case 0: slot = &L.in; N = L.proj_width(); break;
        case 3: slot = &L.out; N = d; K = L.spec.heads * L.spec.vdim; break;
        case 4: slot = &L.gate; N = E * L.spec.ff; break;
        case 5: slot = &L.up; N = E * L.spec.ff; break;
        case 6: slot = &L.down; N = E * d; K = L.spec.ff; break;
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
        AB2_REQUIRE(layer < st->cfg.n_layers && which >= 0 && which <= 4, AB2_ERR_BAD_ARG, "layer %d / norm %d out of range", layer, which);
        StackLayer &L = st->layers[layer];
        AB2_REQUIRE(which != 2 || L.spec.mixer != AB2_MIX_ATTENTION, AB2_ERR_BAD_ARG, "layer %d has no norm inside its mixer", layer);
        float **slots[] = {&L.norm1, &L.norm2, &L.mix_norm, &L.pre1, &L.pre2};
        slot = slots[which];
        if (which == 2) n = L.spec.mixer == AB2_MIX_LATENT ? (size_t)L.spec.kv_rank : (size_t)L.spec.heads * L.spec.vdim;
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

// Routing arrays of a layer with experts by token id, in a block of 2 max_tokens top + 2 (experts + 1) ints.
static MoeRoute table_route(const ab2_layer_spec &sp, int *block, int max_tokens, int T) {
    MoeRoute r = {};
    r.E = sp.experts; r.top = sp.top; r.pairs = T * sp.top;
    r.perm = block; r.expert = r.perm + (size_t)max_tokens * sp.top; r.offset = r.expert + (size_t)max_tokens * sp.top; r.active = r.offset + sp.experts + 1;
    return r;
}

int stack_finalize(Stack *st) {
    const size_t T = st->max_tokens, esz = dtype_size(st->dtype), d = st->cfg.d_model;
    const bool pre = st->form.pre_norms, loops = st->form.loop_times > 0;
    AB2_REQUIRE(st->embedding && (st->embed_norm || !st->form.embed_norm) && st->final_norm, AB2_ERR_BAD_ARG, "embedding or a model-level norm not set");
    AB2_REQUIRE(!loops || st->loop_steps, AB2_ERR_BAD_ARG, "the loop's step vectors are not set");
    if (!st->lm_head) {
        AB2_REQUIRE(st->cfg.tied, AB2_ERR_BAD_ARG, "lm_head not set and embeddings are not tied");
        st->lm_head = st->embedding;
    }
    size_t proj = 0, mixed = 0, mix32 = 0, parts = 1, act = 0, gathered = 0, z = 0, vf = 0, pairs = 0, experts = 0, state = 0, zw = 0, shared = 0, latent = 0, table_layers = 0;
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
        } else if (sp.mixer == AB2_MIX_LATENT) {
            AB2_REQUIRE(L.ukv && L.mix_norm, AB2_ERR_BAD_ARG, "layer %d: the latent's up projection or norm is not set", i);
            if (sp.rot_dims > 0) STEP(rotation_tables(st, sp.rot_dims, sp.rot_base, &L.cos_t, &L.sin_t));
            if (!L.absorb) AB2_CUDA(cudaMalloc((void **)&L.absorb, (size_t)sp.heads * sp.kv_rank * sp.dim * 2));
            STEP(latent_absorb_weights((const __nv_bfloat16 *)L.ukv->codes, L.absorb, sp.heads, sp.dim, sp.vdim, sp.kv_rank, nullptr));
            latent = std::max(latent, latent_workspace(sp.heads, sp.dim, sp.rot_dims, sp.kv_rank, sp.vdim, st->max_tokens, st->cfg.max_seq, st->dtype));
        } else {
            if (sp.rot_dims > 0) STEP(rotation_tables(st, sp.rot_dims, sp.rot_base, &L.cos_t, &L.sin_t));
            if (sp.v_mix) vf = std::max(vf, (size_t)sp.kv_heads * sp.vdim);
        }
        if (sp.ffn == AB2_FFN_MOE) {
            AB2_REQUIRE(L.gate && L.up && L.down && L.norm2 && (sp.routing == AB2_ROUTE_TABLE ? L.table != nullptr : L.router != nullptr), AB2_ERR_BAD_ARG,
                        "layer %d: a weight or norm of the feed-forward is not set", i);
            AB2_REQUIRE(sp.shared_ff == 0 || (L.shared_gate && L.shared_up && L.shared_down), AB2_ERR_BAD_ARG, "layer %d: a weight of the shared expert is not set", i);
            shared = std::max(shared, (size_t)sp.shared_ff);
            table_layers += sp.routing == AB2_ROUTE_TABLE;
            parts = std::max(parts, (size_t)sp.top);
            act = std::max(act, (size_t)sp.top * sp.ff);
            gathered = std::max(gathered, (size_t)sp.top * d);
            z = std::max(z, (size_t)sp.experts);
            pairs = std::max(pairs, (size_t)sp.top);
            experts = std::max(experts, (size_t)sp.experts);
        } else if (sp.ffn == AB2_FFN_POLY) {
            AB2_REQUIRE(L.up && L.down && L.norm2, AB2_ERR_BAD_ARG, "layer %d: a weight or norm of the feed-forward is not set", i);
            zw = std::max(zw, (size_t)sp.ff);
            act = std::max(act, (size_t)sp.ff);
        }
        AB2_REQUIRE(!pre || (L.pre1 && (L.pre2 || sp.ffn == AB2_FFN_NONE)), AB2_ERR_BAD_ARG, "layer %d: a norm before a sublayer is not set", i);
    }
    st->latent_bytes = latent;
    const int n_tables = (int)table_layers;
    if (!st->x) {
        const bool b16 = st->dtype != AB2_F32;
        struct { void **p; size_t bytes; } all[] = {
            {(void **)&st->x, T * d * 4}, {&st->xb, b16 || pre ? T * d * esz : 0}, {&st->proj, T * proj * esz}, {&st->mixed, T * mixed * esz},
            {(void **)&st->mix32, T * mix32 * 4}, {(void **)&st->parts, T * parts * d * 4}, {&st->act, T * act * esz},
            {&st->gathered, b16 ? T * gathered * esz : 0}, {(void **)&st->router_z, T * z * 4}, {&st->v_first, T * vf * esz},
            {&st->head_in, T * d * esz}, {(void **)&st->route_int, (T * pairs * 2 + 2 * (experts + 1)) * 4},
            {(void **)&st->route_score, T * pairs * 4}, {(void **)&st->logits_scratch, T * st->cfg.vocab * 4}, 
            {(void **)&st->seg_states, b16 ? LIGHTNING_MAX_SEGMENTS * state * 4 : 0}, {(void **)&st->x0, st->form.loop_times > 1 ? T * d * 4 : 0},
            {(void **)&st->shared_out, shared ? T * d * 4 : 0}, {&st->shared_act, T * shared * esz}, {&st->z, T * zw * esz},
            {&st->latent_work, latent}, {(void **)&st->route_tables, table_layers * sizeof(MoeTable)}};
        for (auto &a : all) {
            if (a.bytes == 0) continue;
            cudaError_t e = cudaMalloc(a.p, a.bytes);
            if (e != cudaSuccess) {
                free_workspace(st);
                return fail(AB2_ERR_CUDA, "workspace allocation of %zu bytes failed: %s", a.bytes, cudaGetErrorString(e));
            }
        }
    }
    std::vector<MoeTable> tables;
    for (auto &L : st->layers) {
        const ab2_layer_spec &sp = L.spec;
        if (sp.ffn != AB2_FFN_MOE || sp.routing != AB2_ROUTE_TABLE) continue;
        if (!L.route_int) AB2_CUDA(cudaMalloc((void **)&L.route_int, (2 * T * sp.top + 2 * (sp.experts + 1)) * 4));
        tables.push_back({L.table, table_route(L.spec, L.route_int, st->max_tokens, 0)});
    }
    st->n_route_tables = n_tables;
    if (n_tables) AB2_CUDA(cudaMemcpy(st->route_tables, tables.data(), tables.size() * sizeof(MoeTable), cudaMemcpyHostToDevice));
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
        const ab2_layer_spec &sp = st->layers[st->runs[i].layer].spec;
        const bool rec = sp.mixer == AB2_MIX_LIGHTNING;
        if (sp.mixer == AB2_MIX_LATENT) {
            AB2_REQUIRE(!l.recurrent && l.kvh == 1 && l.kd == sp.kv_rank + sp.rot_dims && l.vd == 0 && l.cap == kv->cap && kv->part_acc_bytes >= latent_part_bytes(sp),
                        AB2_ERR_BAD_SHAPE, "cache layer %d does not match the model", i);
            continue;
        }
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

static int latent_mixer(Stack *st, StackLayer &L, ab2_kv *kv, int run, int S, int row0, int nrows, int max_len, cudaStream_t s) {
    const ab2_layer_spec &sp = L.spec;
    LatentArgs a = {};
    a.kv = kv_layer_view(kv, run);
    a.proj = st->proj; a.stride = L.proj_width(); a.S = S; a.row0 = row0; a.H = sp.heads; a.dim = sp.dim; a.rot = sp.rot_dims; a.rank = sp.kv_rank;
    a.vdim = sp.vdim; a.gated = sp.head_gate; a.norm_w = L.mix_norm; a.eps = st->cfg.rms_eps; a.scale = sp.scale; a.cos_t = L.cos_t; a.sin_t = L.sin_t;
    a.ukv = (const __nv_bfloat16 *)L.ukv->codes; a.absorb = L.absorb; a.out = st->mixed; a.work = st->latent_work; a.work_bytes = st->latent_bytes;
    return latent_attention(kv, a, nrows, max_len, st->dtype, s);
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
    STEP(linear_moe_glu(gate, up, in, dtype, w.act, sp.glu, sp.limit, true, r, w.gathered, s));
    return linear_moe_down(down, w.act, dtype, parts, 1.f, r, s);
}

// st->parts [T][top][d] and, with a shared expert, st->shared_out [T][d]
static int moe_ffn(Stack *st, StackLayer &L, const void *in, int T, cudaStream_t s) {
    const ab2_layer_spec &sp = L.spec;
    if (sp.shared_ff > 0) {
        STEP(linear_glu(L.shared_gate, L.shared_up, in, T, st->dtype, st->shared_act, sp.glu, sp.limit, s));
        STEP(linear_bf16(L.shared_down, st->shared_act, T, st->dtype, st->shared_out, LIN_F32, 0, s));
    }
    if (sp.routing == AB2_ROUTE_TABLE) {
        const MoeRoute r = table_route(sp, L.route_int, st->max_tokens, T);
        STEP(linear_moe_glu(L.gate, L.up, in, st->dtype, st->act, sp.glu, sp.limit, false, r, st->gathered, s));
        return linear_moe_down(L.down, st->act, st->dtype, st->parts, 1.f / (float)sp.top, r, s);
    }
    const MoeScratch w = {st->router_z, st->route_int, st->route_score, st->act, st->gathered};
    return moe_experts(sp, L.router, L.gate, L.up, L.down, in, T, st->dtype, w, st->parts, s);
}

static int poly_ffn(Stack *st, StackLayer &L, const void *in, int T, cudaStream_t s) {
    const ab2_layer_spec &sp = L.spec;
    PolyNormArgs p = {st->z, st->act, sp.ff, sp.poly[0], sp.poly[1], sp.poly[2], sp.poly[3], st->cfg.rms_eps};
    STEP(linear_bf16(L.up, in, T, st->dtype, st->z, LIN_STORE, 0, s));
    STEP(launch_poly_norm(p, T, st->dtype, s));
    return linear_bf16(L.down, st->act, T, st->dtype, st->parts, LIN_F32, 0, s);
}

int stack_forward(Stack *st, ab2_kv *kv, const uint32_t *ids, int S, int row0, int nrows, int logits_mode, float *logits,
                  uint32_t *argmax_out, int len_hint, cudaStream_t s) {
    const int T = nrows * S, d = st->cfg.d_model;
    int max_len = len_hint;
    if (max_len <= 0)
        for (int i = 0; i < nrows; ++i) max_len = std::max(max_len, kv->lens_host[kv_row_host(kv, row0, i)] + S);
    const bool pre = st->form.pre_norms;
    const void *in = st->dtype == AB2_F32 && !pre ? (const void *)st->x : st->xb;  // what the sublayers read
    const int n_runs = (int)st->runs.size();
    ResidualNormArgs n = {};
    n.eps = st->cfg.rms_eps; n.d = d; n.x = st->x; n.out = st->xb;
    // what comes between a sublayer and the first of run r: the start of a pass, the norm before the sublayer
    auto enter = [&](int r) {
        n.add = nullptr; n.x0 = nullptr; n.w_next = nullptr;
        if (r == n_runs) return;
        const Stack::Run &run = st->runs[r];
        if (run.pass >= 0) n.add = st->loop_steps + (size_t)run.pass * d;
        if (run.pass > 0) n.x0 = st->x0;
        if (pre) n.w_next = st->layers[run.layer].pre1;
    };
    if (st->n_route_tables) STEP(moe_route_tables(st->route_tables, st->n_route_tables, ids, st->cfg.vocab, T, s));
    enter(0);
    n.w = st->form.embed_norm ? st->embed_norm : nullptr; n.table = (const __nv_bfloat16 *)st->embedding->codes; n.ids = ids; n.vocab = st->cfg.vocab;
    n.x0 = st->form.loop_times > 1 ? st->x0 : nullptr;
    STEP(launch_residual_norm(n, RN_EMBED, T, st->dtype, s));
    const bool want_logits = logits_mode != 0 || argmax_out != nullptr, last = logits_mode != 2;
    const bool final_norm_rides = pre && want_logits && (!last || S == 1);  // the last sublayer's norm kernel makes the head's input
    for (int r = 0; r < n_runs; ++r) {
        StackLayer &L = st->layers[st->runs[r].layer];
        const ab2_layer_spec &sp = L.spec;
        auto end_of_run = [&]() {
            enter(r + 1);
            if (r + 1 == n_runs && pre) { n.w_next = st->final_norm; n.out = final_norm_rides ? st->head_in : nullptr; }
        };
        if (sp.mixer == AB2_MIX_LIGHTNING) {
            STEP(linear_bf16(L.in, in, T, st->dtype, st->proj, LIN_ACT, sp.heads * (2 * sp.dim + sp.vdim), s));
            STEP(lightning_mixer(st, L, kv, r, S, row0, nrows, s));
        } else {
            STEP(linear_bf16(L.in, in, T, st->dtype, st->proj, LIN_STORE, 0, s));
            if (sp.mixer == AB2_MIX_LATENT) STEP(latent_mixer(st, L, kv, r, S, row0, nrows, max_len, s));
            else STEP(attention_mixer(st, L, kv, r, S, row0, nrows, max_len, s));
        }
        STEP(linear_bf16(L.out, st->mixed, T, st->dtype, st->parts, LIN_F32, 0, s));
        n.w = L.norm1; n.parts = st->parts; n.nparts = 1; n.extra = nullptr;
        if (sp.ffn == AB2_FFN_NONE) end_of_run();
        else { n.add = nullptr; n.x0 = nullptr; n.w_next = pre ? L.pre2 : nullptr; }
        STEP(launch_residual_norm(n, RN_ADD, T, st->dtype, s));
        if (sp.ffn == AB2_FFN_NONE) continue;
        STEP(sp.ffn == AB2_FFN_MOE ? moe_ffn(st, L, in, T, s) : poly_ffn(st, L, in, T, s));
        n.w = L.norm2; n.nparts = sp.ffn == AB2_FFN_MOE ? sp.top : 1;
        n.extra = sp.ffn == AB2_FFN_MOE && sp.shared_ff > 0 ? st->shared_out : nullptr;
        end_of_run();
        STEP(launch_residual_norm(n, RN_ADD, T, st->dtype, s));
    }
    if (!want_logits) return AB2_OK;
    const int rows = last ? nrows : T;
    AB2_REQUIRE(!argmax_out || last || S == 1, AB2_ERR_UNSUPPORTED, "argmax with all-token logits needs S == 1");
    if (!final_norm_rides) {
        n.w = st->final_norm; n.step = last ? S : 1; n.out = st->head_in;
        STEP(launch_residual_norm(n, RN_FINAL, rows, st->dtype, s));
    }
    float *lg = logits ? logits : st->logits_scratch;
    LinArgs head = {};
    head.w = (const __nv_bfloat16 *)st->lm_head->codes; head.x = st->head_in; head.y = lg; head.N = st->lm_head->N; head.K = st->lm_head->K; head.M = rows;
    head.ldx = head.K; head.ldy = head.N; head.batch = 1; head.epi = LIN_F32; head.cap = st->form.logit_softcap;
    STEP(linear_dense(head, st->dtype, s));
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
    if (mixer != AB2_MIX_LIGHTNING) STEP(check_spec(*spec, layer));
    const KvLayer &l = kv->layers[layer];
    const bool rec = mixer == AB2_MIX_LIGHTNING;
    if (mixer == AB2_MIX_LATENT)
        AB2_REQUIRE(!l.recurrent && l.kvh == 1 && l.kd == spec->kv_rank + spec->rot_dims && l.vd == 0 && kv->part_acc_bytes >= latent_part_bytes(*spec),
                    AB2_ERR_BAD_SHAPE, "cache layer %d does not match the spec", layer);
    else
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

AB2_API int ab2_latent_workspace(const ab2_layer_spec *spec, int tokens, int positions, ab2_dtype dtype, size_t *bytes) {
    AB2_REQUIRE(spec && bytes, AB2_ERR_BAD_ARG, "null argument");
    STEP(check_spec(*spec, 0));
    AB2_REQUIRE(spec->mixer == AB2_MIX_LATENT && tokens > 0 && positions > 0, AB2_ERR_BAD_ARG, "a latent mixer and positive sizes expected");
    *bytes = up256((size_t)spec->heads * spec->kv_rank * spec->dim * 2) +
             latent_workspace(spec->heads, spec->dim, spec->rot_dims, spec->kv_rank, spec->vdim, tokens, positions, dtype);
    return AB2_OK;
}

AB2_API int ab2_latent_attention(ab2_kv *kv, int layer, const ab2_layer_spec *spec, void *proj_dev, long long stride, const float *norm_dev,
                                 const ab2_qweight *ukv, const float *cos_dev, const float *sin_dev, float eps, void *out_dev,
                                 void *workspace_dev, size_t workspace_bytes, int reuse, int S, int row0, int nrows, ab2_dtype dtype, ab2_stream stream) {
    STEP(check_mixer_call(kv, layer, spec, AB2_MIX_LATENT, proj_dev, out_dev, S, row0, nrows, dtype));
    const int H = spec->heads, D = spec->dim + spec->rot_dims;
    AB2_REQUIRE(norm_dev && ukv && workspace_dev && (spec->rot_dims == 0 || (cos_dev && sin_dev)), AB2_ERR_BAD_ARG, "null argument");
    AB2_REQUIRE(ukv->fmt == FMT_BF16 && ukv->N == H * (spec->dim + spec->vdim) && ukv->K == spec->kv_rank, AB2_ERR_BAD_SHAPE, "the up projection does not match the spec");
    AB2_REQUIRE(stride >= (long long)H * D + spec->kv_rank + spec->rot_dims + (spec->head_gate ? H : 0), AB2_ERR_BAD_SHAPE, "row stride %lld is too short", stride);
    const size_t absorb = up256((size_t)H * spec->kv_rank * spec->dim * 2);  // the transposed weight comes first
    AB2_REQUIRE(workspace_bytes >= absorb + latent_workspace(H, spec->dim, spec->rot_dims, spec->kv_rank, spec->vdim, nrows * S, 1, dtype), AB2_ERR_BAD_SHAPE,
                "workspace of %zu bytes is too small", workspace_bytes);
    __nv_bfloat16 *absorbed = (__nv_bfloat16 *)workspace_dev;
    if (!reuse) STEP(latent_absorb_weights((const __nv_bfloat16 *)ukv->codes, absorbed, H, spec->dim, spec->vdim, spec->kv_rank, (cudaStream_t)stream));
    LatentArgs a = {};
    a.kv = kv_layer_view(kv, layer);
    a.proj = proj_dev; a.stride = stride; a.S = S; a.row0 = row0; a.H = H; a.dim = spec->dim; a.rot = spec->rot_dims; a.rank = spec->kv_rank;
    a.vdim = spec->vdim; a.gated = spec->head_gate; a.norm_w = norm_dev; a.eps = eps; a.scale = spec->scale; a.cos_t = cos_dev; a.sin_t = sin_dev;
    a.ukv = (const __nv_bfloat16 *)ukv->codes; a.absorb = absorbed; a.out = out_dev; a.work = (char *)workspace_dev + absorb; a.work_bytes = workspace_bytes - absorb;
    int max_len = 0;
    for (int i = 0; i < nrows; ++i) max_len = std::max(max_len, kv->lens_host[row0 + i] + S);
    return latent_attention(kv, a, nrows, max_len, dtype, (cudaStream_t)stream);
}

AB2_API int ab2_poly_norm(const void *z_dev, void *out_dev, int rows, int n, const float *coef_host, float eps, ab2_dtype dtype, ab2_stream stream) {
    AB2_REQUIRE(z_dev && out_dev && coef_host, AB2_ERR_BAD_ARG, "null argument");
    AB2_REQUIRE(rows > 0 && n > 0, AB2_ERR_BAD_SHAPE, "%d rows of %d values", rows, n);
    AB2_REQUIRE(dtype == AB2_F32 || dtype == AB2_BF16, AB2_ERR_BAD_DTYPE, "unsupported dtype %d", (int)dtype);
    const PolyNormArgs p = {z_dev, out_dev, n, coef_host[0], coef_host[1], coef_host[2], coef_host[3], eps};
    return launch_poly_norm(p, rows, dtype, (cudaStream_t)stream);
}

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
