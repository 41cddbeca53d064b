// Latent attention: what a token leaves in the cache is one latent c of `rank` values and one rotated key
// part that all heads share; head h's key is (W_uk,h c, key part) and its value W_uv,h c.
//
//   latent_prep_kernel     norm of the latent, rotation of queries and key part, store into the cache
//   latent_absorb_kernel   the same and the queries against the latents, in one launch (bf16)
//   latent_tc_kernel       attention in the latent space on the tensor cores (attention_latent_tc.cu)
//   latent_attn_kernel     the same on CUDA cores: f32 models, latents that shared memory cannot hold
//   latent_merge_kernel    merge of the splits of a query's keys
//
// Decoding and short portions of a prompt never form keys and values: W_uk,h^T q_h is a query against
// the latents themselves ("absorbed"), the softmax weights sum latents, and W_uv,h turns the sum
// into the head's output.  Longer portions project the cached latents to keys and values once, some
// heads at a time, and run prompt_attention over them.
// Scores, softmax weights and sums are f32 throughout.
#include <algorithm>
#include <cfloat>

#include "stack.cuh"

using namespace ab2;

namespace ab2 {
int device_sm_count();
namespace {

// One CTA per token.  Rotated queries go to `qx` ([token][H][kds], behind the latent part; the padding is
// zeroed) or stay where they are (qx null).
template <typename T>
__global__ void __launch_bounds__(256) latent_prep_kernel(LatentArgs a, T *qx) {
    __shared__ float warp_sums[8];
    pdl_wait();
    pdl_launch_dependents();
    const KvLayer &l = a.kv.l;
    const int s = blockIdx.x, rrow = blockIdx.y, row = kv_row(a.kv, a.row0, rrow), pos = a.kv.lens[row] + s;
    const size_t tok = (size_t)rrow * a.S + s;
    T *q = (T *)a.proj + tok * a.stride;
    const T *c = q + (size_t)a.H * (a.dim + a.rot), *kr = c + a.rank;
    T *dst = (T *)l.k + ((size_t)row * l.cap + pos) * l.kds;  // capacity is checked on the host
    const int half = a.rot >> 1;
    const float *ct = a.cos_t + (size_t)pos * half, *st = a.sin_t + (size_t)pos * half;
    float sum = 0.f;
    for (int i = threadIdx.x; i < a.rank; i += 256) {
        const float v = to_f32(c[i]);
        sum = fmaf(v, v, sum);
    }
    // a warp takes every eighth head (the key part counts as the last); a lane keeps its angles for all of them
    struct alignas(2 * sizeof(T)) Pair { T u, v; };
    const bool paired = ((a.dim | (int)a.stride | a.rank) & 1) == 0;  // pairs lie on their own size (rot and kds are even)
    for (int j = threadIdx.x & 31; j < half; j += 32) {
        const float cs = ct[j], sn = st[j];
#pragma unroll 4
        for (int h = threadIdx.x >> 5; h <= a.H; h += 8) {
            const T *src = (h < a.H ? q + (size_t)h * (a.dim + a.rot) + a.dim : kr) + 2 * j;
            T *out = (h == a.H ? dst + a.rank : qx ? qx + (tok * a.H + h) * l.kds + a.rank : q + (size_t)h * (a.dim + a.rot) + a.dim) + 2 * j;
            Pair p;
            if (paired) p = *reinterpret_cast<const Pair *>(src);
            else { p.u = src[0]; p.v = src[1]; }
            const float u = to_f32(p.u), v = to_f32(p.v);
            p.u = from_f32<T>(u * cs - v * sn);
            p.v = from_f32<T>(v * cs + u * sn);
            if (paired) *reinterpret_cast<Pair *>(out) = p;
            else { out[0] = p.u; out[1] = p.v; }
        }
    }
    const int used = a.rank + a.rot, pad = l.kds - used;
    if (qx)
        for (int i = threadIdx.x; i < a.H * pad; i += 256) qx[(tok * a.H + i / pad) * l.kds + used + i % pad] = from_f32<T>(0.f);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    if ((threadIdx.x & 31) == 0) warp_sums[threadIdx.x >> 5] = sum;
    __syncthreads();
    sum = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) sum += warp_sums[w];
    const float inv = 1.f / sqrtf(sum / (float)a.rank + a.eps);
    for (int i = threadIdx.x; i < a.rank; i += 256) dst[i] = from_f32<T>(to_f32(c[i]) * inv * a.norm_w[i]);
}

// grid (nsplit, head groups, nrows * S), 256 threads: REP heads of one query over a run of its keys, 32
// keys at a time through shared memory.  In the score phase a warp takes a key, in the sum phase a
// thread takes up to four latent dimensions.
constexpr int LA_REP = 4, LA_KEYS = 32;

template <typename T>
__global__ void __launch_bounds__(256) latent_attn_kernel(LatentArgs a, const T *qx, T *ox) {
    extern __shared__ __align__(16) float dyn[];
    __shared__ float ps[LA_REP][LA_KEYS], corr[LA_REP], m_run[LA_REP], l_run[LA_REP];
    pdl_wait();
    pdl_launch_dependents();
    const KvLayer &l = a.kv.l;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float *qs = dyn, *ks = dyn + LA_REP * l.kds;
    const int head0 = blockIdx.y * LA_REP, nh = min(LA_REP, a.H - head0);
    const int rrow = blockIdx.z / a.S, qi = blockIdx.z % a.S, row = kv_row(a.kv, a.row0, rrow);
    const int n = a.kv.lens[row] + qi + 1;
    const int per = ((n + a.nsplit - 1) / a.nsplit + LA_KEYS - 1) / LA_KEYS * LA_KEYS;
    const int j0 = (int)blockIdx.x * per, j1 = min(n, j0 + per);
    const T *kb = (const T *)l.k + (size_t)row * l.cap * l.kds;
    const size_t tok = blockIdx.z;
    for (int i = threadIdx.x; i < LA_REP * l.kds; i += 256) qs[i] = i / l.kds < nh ? to_f32(qx[(tok * a.H + head0) * l.kds + i]) : 0.f;
    if (threadIdx.x < LA_REP) { m_run[threadIdx.x] = -INFINITY; l_run[threadIdx.x] = 0.f; }
    float acc[LA_REP][4];
#pragma unroll
    for (int h = 0; h < LA_REP; ++h)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[h][j] = 0.f;
    for (int base = j0; base < j1; base += LA_KEYS) {
        const int nk = min(LA_KEYS, j1 - base);
        __syncthreads();
        for (int i = threadIdx.x; i < nk * l.kds; i += 256) ks[i] = to_f32(kb[(size_t)base * l.kds + i]);
        __syncthreads();
        for (int k = warp; k < LA_KEYS; k += 8) {
            float sc[LA_REP] = {0.f, 0.f, 0.f, 0.f};
            if (k < nk)
                for (int d = lane; d < l.kds; d += 32) {
                    const float kv = ks[k * l.kds + d];
#pragma unroll
                    for (int h = 0; h < LA_REP; ++h) sc[h] = fmaf(qs[h * l.kds + d], kv, sc[h]);
                }
#pragma unroll
            for (int h = 0; h < LA_REP; ++h) {
#pragma unroll
                for (int o = 16; o > 0; o >>= 1) sc[h] += __shfl_xor_sync(0xffffffffu, sc[h], o);
                if (lane == 0) ps[h][k] = k < nk ? sc[h] * a.scale : -INFINITY;
            }
        }
        __syncthreads();
        if (warp < LA_REP) {
            const float s = ps[warp][lane];
            float m = s;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
            const float old = m_run[warp], top = fmaxf(old, m), p = expf(s - top);
            float sum = p;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
            ps[warp][lane] = p;
            if (lane == 0) {
                const float c = expf(old - top);
                corr[warp] = c; m_run[warp] = top; l_run[warp] = l_run[warp] * c + sum;
            }
        }
        __syncthreads();
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int d = threadIdx.x + 256 * j;
            if (d >= a.rank) break;
            float r[LA_REP];
#pragma unroll
            for (int h = 0; h < LA_REP; ++h) r[h] = acc[h][j] * corr[h];
            for (int k = 0; k < nk; ++k) {
                const float v = ks[k * l.kds + d];
#pragma unroll
                for (int h = 0; h < LA_REP; ++h) r[h] = fmaf(ps[h][k], v, r[h]);
            }
#pragma unroll
            for (int h = 0; h < LA_REP; ++h) acc[h][j] = r[h];
        }
    }
    __syncthreads();
#pragma unroll
    for (int h = 0; h < LA_REP; ++h) {
        if (h >= nh) break;
        const size_t r = tok * a.H + head0 + h;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int d = threadIdx.x + 256 * j;
            if (d >= a.rank) break;
            if (a.nsplit == 1) ox[r * a.rank + d] = from_f32<T>(acc[h][j] / l_run[h]);
            else a.part_acc[(r * a.nsplit + blockIdx.x) * a.rank + d] = acc[h][j];
        }
        if (a.nsplit > 1 && threadIdx.x == 0) {
            a.part_ml[(r * a.nsplit + blockIdx.x) * 2] = m_run[h] * 1.44269504088896341f;  // in powers of two
            a.part_ml[(r * a.nsplit + blockIdx.x) * 2 + 1] = l_run[h];
        }
    }
}

// grid (token-head rows, ceil(rank / (1024 / G))): ox = sum of the splits' latents, weighted by 2^(m - max), over
// the sum of their weights.  A thread takes four dimensions of every G-th split, eight splits at most.
template <typename T, int G>
__global__ void __launch_bounds__(256) latent_merge_kernel(LatentArgs a, T *ox) {
    constexpr int LANES = 256 / G;
    __shared__ float wt[AB2_KV_MAX_SPLITS];
    __shared__ float4 red[G][LANES];
    pdl_wait();
    pdl_launch_dependents();
    const int group = threadIdx.x / LANES, lane = threadIdx.x % LANES;
    const size_t r = blockIdx.x, p0 = r * a.nsplit;
    const int d0 = (blockIdx.y * LANES + lane) * 4, nd = min(4, a.rank - d0);
    const float *src = a.part_acc + p0 * a.rank + d0;
    float4 v[8];
#pragma unroll
    for (int k = 0; k < 8; ++k) {
        const int sp = group + G * k;
        v[k] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (sp < a.nsplit && nd == 4 && (a.rank & 3) == 0) v[k] = *reinterpret_cast<const float4 *>(src + (size_t)sp * a.rank);
    }
    if ((a.rank & 3) != 0)
        for (int k = 0; k < 8 && group + G * k < a.nsplit; ++k) {
            const float *q = src + (size_t)(group + G * k) * a.rank;
            if (nd > 0) v[k].x = q[0];
            if (nd > 1) v[k].y = q[1];
            if (nd > 2) v[k].z = q[2];
            if (nd > 3) v[k].w = q[3];
        }
    if (threadIdx.x < 32) {
        float m[2], ls[2], top = -INFINITY, sum = 0.f;
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const int sp = threadIdx.x + 32 * k;
            m[k] = sp < a.nsplit ? a.part_ml[(p0 + sp) * 2] : -INFINITY;
            ls[k] = sp < a.nsplit ? a.part_ml[(p0 + sp) * 2 + 1] : 0.f;
            top = fmaxf(top, m[k]);
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, o));
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            m[k] = m[k] == -INFINITY ? 0.f : exp2f(m[k] - top);
            sum = fmaf(m[k], ls[k], sum);
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
#pragma unroll
        for (int k = 0; k < 2; ++k) wt[threadIdx.x + 32 * k] = m[k] / sum;
    }
    __syncthreads();
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int k = 0; k < 8; ++k) {
        const float w = group + G * k < a.nsplit ? wt[group + G * k] : 0.f;
        if (w != 0.f) {  // an empty split has written nothing
            s.x = fmaf(w, v[k].x, s.x); s.y = fmaf(w, v[k].y, s.y); s.z = fmaf(w, v[k].z, s.z); s.w = fmaf(w, v[k].w, s.w);
        }
    }
    if (G > 1) {
        red[group][lane] = s;
        __syncthreads();
        if (group > 0) return;
#pragma unroll
        for (int g = 1; g < G; ++g) {
            const float4 q = red[g][lane];
            s.x += q.x; s.y += q.y; s.z += q.z; s.w += q.w;
        }
    }
    T *dst = ox + r * a.rank + d0;
    if (nd > 0) dst[0] = from_f32<T>(s.x);
    if (nd > 1) dst[1] = from_f32<T>(s.y);
    if (nd > 2) dst[2] = from_f32<T>(s.z);
    if (nd > 3) dst[3] = from_f32<T>(s.w);
}

template <typename T>
cudaError_t launch_merge(const LatentArgs &a, T *ox, int rows, cudaStream_t s) {
    if (a.nsplit <= 8 && a.rank > 256) return launch_kernel(latent_merge_kernel<T, 1>, dim3(rows, (a.rank + 1023) / 1024), dim3(256), 0, s, a, ox);
    if (a.nsplit <= 16) return launch_kernel(latent_merge_kernel<T, 2>, dim3(rows, (a.rank + 511) / 512), dim3(256), 0, s, a, ox);
    return launch_kernel(latent_merge_kernel<T, 8>, dim3(rows, (a.rank + 127) / 128), dim3(256), 0, s, a, ox);
}

// bf16, few tokens: absorbed queries, rotations, norm and store in one launch.  grid (ceil(rank / 128), token
// tiles of 8 NT, H + 1), 256 threads.  A layer z < H of the grid multiplies W_uk,h^T by the head's unrotated
// queries: a warp owns 16 latent dimensions over the whole (short) sum, its fragments read as in
// gemv_bf16.cu; its first CTA rotates the head's queries.  Layer H norms the latents, rotates the key
// parts and stores both.  KC chunks of 32 unrotated dimensions.
__device__ __forceinline__ void mma_bf16(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

template <int KC, int NT>
__global__ void __launch_bounds__(256) latent_absorb_kernel(LatentArgs a, __nv_bfloat16 *qx, int tokens) {
    __shared__ __align__(16) __nv_bfloat16 tile[8 * NT][128 + 8];
    const KvLayer &l = a.kv.l;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, c = lane & 3;
    const int h = blockIdx.z, m0 = blockIdx.y * 8 * NT, r0 = blockIdx.x * 128, D = a.dim + a.rot, half = a.rot >> 1;
    const __nv_bfloat16 *proj = (const __nv_bfloat16 *)a.proj;
    auto position = [&](int t, int &row) {
        row = kv_row(a.kv, a.row0, t / a.S);
        return a.kv.lens[row] + t % a.S;
    };
    if (h == a.H) {
        pdl_wait();
        pdl_launch_dependents();
        for (int t = m0 + blockIdx.x * 8 + warp; t < min(tokens, m0 + 8 * NT); t += 8 * gridDim.x) {
            int row;
            const int pos = position(t, row);
            const __nv_bfloat16 *src = proj + t * a.stride + (size_t)a.H * D;
            __nv_bfloat16 *dst = (__nv_bfloat16 *)l.k + ((size_t)row * l.cap + pos) * l.kds;  // capacity is checked on the host
            uint4 v[4];  // a lane's values, eight at a time; rank is a multiple of 8 and 1024 at most
#pragma unroll
            for (int k = 0; k < 4; ++k) v[k] = (lane + 32 * k) * 8 < a.rank ? reinterpret_cast<const uint4 *>(src)[lane + 32 * k] : make_uint4(0u, 0u, 0u, 0u);
            float sum = 0.f;
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const uint32_t w[4] = {v[k].x, v[k].y, v[k].z, v[k].w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float lo = __uint_as_float(w[e] << 16), hi = __uint_as_float(w[e] & 0xffff0000u);
                    sum = fmaf(lo, lo, fmaf(hi, hi, sum));
                }
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
            const float inv = 1.f / sqrtf(sum / (float)a.rank + a.eps);
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const int d = (lane + 32 * k) * 8;
                if (d >= a.rank) continue;
                const float4 na = reinterpret_cast<const float4 *>(a.norm_w + d)[0], nb = reinterpret_cast<const float4 *>(a.norm_w + d)[1];
                const uint32_t w[4] = {v[k].x, v[k].y, v[k].z, v[k].w};
                const float nw[8] = {na.x, na.y, na.z, na.w, nb.x, nb.y, nb.z, nb.w};
                uint32_t o[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const __nv_bfloat162 q = __floats2bfloat162_rn(__uint_as_float(w[e] << 16) * inv * nw[2 * e], __uint_as_float(w[e] & 0xffff0000u) * inv * nw[2 * e + 1]);
                    o[e] = *reinterpret_cast<const uint32_t *>(&q);
                }
                *reinterpret_cast<uint4 *>(dst + d) = make_uint4(o[0], o[1], o[2], o[3]);
            }
            for (int j = lane; j < half; j += 32) {
                const float u = __bfloat162float(src[a.rank + 2 * j]), v = __bfloat162float(src[a.rank + 2 * j + 1]);
                const float cs = a.cos_t[(size_t)pos * half + j], sn = a.sin_t[(size_t)pos * half + j];
                dst[a.rank + 2 * j] = __float2bfloat16_rn(u * cs - v * sn);
                dst[a.rank + 2 * j + 1] = __float2bfloat16_rn(v * cs + u * sn);
            }
        }
        return;
    }
    const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
    const int ra = r0 + warp * 16 + g;
    const __nv_bfloat16 *w = a.absorb + (size_t)h * a.rank * a.dim + c * 8;
    uint4 va[KC], vb[KC];
#pragma unroll
    for (int k = 0; k < KC; ++k) {
        const bool in = k * 32 + c * 8 < a.dim;  // dim is a multiple of 8
        va[k] = in ? *reinterpret_cast<const uint4 *>(w + (size_t)min(ra, a.rank - 1) * a.dim + k * 32) : zero;
        vb[k] = in ? *reinterpret_cast<const uint4 *>(w + (size_t)min(ra + 8, a.rank - 1) * a.dim + k * 32) : zero;
    }
    pdl_wait();
    pdl_launch_dependents();
    float acc[NT][4];
#pragma unroll
    for (int j = 0; j < NT; ++j) {
        acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
        const int t = m0 + j * 8 + g;
        const __nv_bfloat16 *x = proj + (size_t)min(t, tokens - 1) * a.stride + (size_t)h * D + c * 8;
#pragma unroll
        for (int k = 0; k < KC; ++k) {
            const uint4 b = k * 32 + c * 8 < a.dim ? *reinterpret_cast<const uint4 *>(x + k * 32) : zero;
            mma_bf16(acc[j], va[k].x, vb[k].x, va[k].y, vb[k].y, b.x, b.y);
            mma_bf16(acc[j], va[k].z, vb[k].z, va[k].w, vb[k].w, b.z, b.w);
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) tile[j * 8 + 2 * c + (i & 1)][warp * 16 + g + 8 * (i >> 1)] = __float2bfloat16_rn(acc[j][i]);
    }
    // this head's queries, rotated behind the latent part, and the padding of a row: the CTAs of a head share its tokens
    const int pairs = half + ((l.kds - a.rank - a.rot) >> 1);  // rotated ones, then padding (rank, rot and kds are even)
    for (int i = blockIdx.x * 256 + threadIdx.x; i < 8 * NT * pairs; i += 256 * gridDim.x) {
        const int t = m0 + i / pairs, j = i % pairs;
        if (t >= tokens) break;
        float u = 0.f, v = 0.f, cs = 0.f, sn = 0.f;
        if (j < half) {
            int row;
            const int pos = position(t, row);
            const __nv_bfloat162 q = *reinterpret_cast<const __nv_bfloat162 *>(proj + t * a.stride + (size_t)h * D + a.dim + 2 * j);
            u = __low2float(q); v = __high2float(q); cs = a.cos_t[(size_t)pos * half + j]; sn = a.sin_t[(size_t)pos * half + j];
        }
        *reinterpret_cast<__nv_bfloat162 *>(qx + ((size_t)t * a.H + h) * l.kds + a.rank + 2 * j) = __floats2bfloat162_rn(u * cs - v * sn, v * cs + u * sn);
    }
    __syncthreads();
    for (int i = threadIdx.x; i < 8 * NT * 16; i += 256) {  // 8 dimensions each
        const int t = m0 + i / 16, d = r0 + (i % 16) * 8;
        if (t < tokens && d < a.rank) *reinterpret_cast<uint4 *>(qx + ((size_t)t * a.H + h) * l.kds + d) = *reinterpret_cast<const uint4 *>(&tile[i / 16][(i % 16) * 8]);
    }
}

template <int KC>
cudaError_t launch_absorb(const LatentArgs &a, __nv_bfloat16 *qx, int tokens, cudaStream_t s) {
    const int nt = tokens <= 8 ? 1 : tokens <= 16 ? 2 : 4;
    const dim3 grid((a.rank + 127) / 128, (tokens + 8 * nt - 1) / (8 * nt), a.H + 1);
    if (nt == 1) return launch_kernel(latent_absorb_kernel<KC, 1>, grid, dim3(256), 0, s, a, qx, tokens);
    if (nt == 2) return launch_kernel(latent_absorb_kernel<KC, 2>, grid, dim3(256), 0, s, a, qx, tokens);
    return launch_kernel(latent_absorb_kernel<KC, 4>, grid, dim3(256), 0, s, a, qx, tokens);
}

__global__ void absorb_weights_kernel(const __nv_bfloat16 *ukv, __nv_bfloat16 *absorb, int dim, int vdim, int rank) {
    __shared__ __nv_bfloat16 tile[32][33];
    const int h = blockIdx.z, r0 = blockIdx.x * 32, d0 = blockIdx.y * 32;
    const __nv_bfloat16 *src = ukv + (size_t)h * (dim + vdim) * rank;
    __nv_bfloat16 *dst = absorb + (size_t)h * rank * dim;
    for (int i = threadIdx.y; i < 32; i += 8)
        if (d0 + i < dim && r0 + threadIdx.x < rank) tile[i][threadIdx.x] = src[(size_t)(d0 + i) * rank + r0 + threadIdx.x];
    __syncthreads();
    for (int i = threadIdx.y; i < 32; i += 8)
        if (r0 + i < rank && d0 + threadIdx.x < dim) dst[(size_t)(r0 + i) * dim + d0 + threadIdx.x] = tile[threadIdx.x][i];
}

size_t up256(size_t n) { return (n + 255) / 256 * 256; }
int row_stride(int rank, int rot) { return (rank + rot + 7) / 8 * 8; }

// Portions from this many tokens on project the latents to keys and values.
constexpr int EXPAND_TOKENS = 128;

bool expandable(int dim, int rot, int rank, int vdim, ab2_dtype dtype) {
    return dtype == AB2_BF16 && rank % 8 == 0 && prompt_attention_serves(dim, rot, vdim);
}

// Attention of a.S queries per row in the latent space: qx [T][H][kds] -> ox [T][H][rank].
template <typename T>
int latent_space_attention(const ab2_kv *kv, LatentArgs a, const T *qx, T *ox, int nrows, int max_len, cudaStream_t s) {
    const KvLayer &l = a.kv.l;
    if (sizeof(T) == 2 && latent_tc_serves(a.rank, l.kds)) {
        int rc = latent_tc_attention(a, (const __nv_bfloat16 *)qx, (__nv_bfloat16 *)ox, kv->B, nrows, max_len, s);
        if (rc != AB2_OK || a.nsplit == 1) return rc;
        cudaError_t e = launch_merge<T>(a, ox, nrows * a.S * a.H, s);
        if (e != cudaSuccess) return fail(AB2_ERR_CUDA, "latent attention launch failed: %s", cudaGetErrorString(e));
        return AB2_OK;
    }
    const int tokens = nrows * a.S, groups = (a.H + LA_REP - 1) / LA_REP, units = groups * tokens;
    a.nsplit = 1;
    if (units < device_sm_count()) {  // the splits' sums fit the scratch: LATENT_PART_TILES * LATENT_ROWS rows
        const int fit = LATENT_PART_TILES * LATENT_ROWS / (tokens * a.H);
        a.nsplit = std::max(1, std::min(std::min(2 * device_sm_count() / units, (max_len + 127) / 128), std::min(fit, AB2_KV_MAX_SPLITS)));
    }
    const size_t smem = (size_t)(LA_REP + LA_KEYS) * l.kds * 4;
    AB2_REQUIRE(smem <= 200 * 1024, AB2_ERR_UNSUPPORTED, "latent rows of %d values exceed shared memory", l.kds);
    static bool configured[64] = {false};  // the attribute is per device (and per T)
    int dev = 0;
    AB2_CUDA(cudaGetDevice(&dev));
    AB2_REQUIRE(dev >= 0 && dev < 64, AB2_ERR_BAD_ARG, "device index %d out of range", dev);
    if (!configured[dev]) {
        AB2_CUDA(cudaFuncSetAttribute(latent_attn_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
        configured[dev] = true;
    }
    cudaError_t e = launch_kernel(latent_attn_kernel<T>, dim3(a.nsplit, groups, tokens), dim3(256), smem, s, a, qx, ox);
    if (e == cudaSuccess && a.nsplit > 1) e = launch_merge<T>(a, ox, tokens * a.H, s);
    if (e != cudaSuccess) return fail(AB2_ERR_CUDA, "latent attention launch failed: %s", cudaGetErrorString(e));
    return AB2_OK;
}

template <typename T>
int launch_latent(const ab2_kv *kv, LatentArgs a, int nrows, int max_len, ab2_dtype dtype, cudaStream_t s) {
    const KvLayer &l = a.kv.l;
    const int T_ = nrows * a.S, D = a.dim + a.rot;
    const T *gate = a.gated ? (const T *)a.proj + (size_t)a.H * D + a.rank + a.rot : nullptr;
    const size_t head_bytes = (size_t)max_len * (a.dim + a.vdim) * 2;  // keys and values of one head
    const bool expand = a.S >= EXPAND_TOKENS && expandable(a.dim, a.rot, a.rank, a.vdim, dtype) && D % 2 == 0 && a.stride % 8 == 0 && a.work_bytes >= head_bytes;
    T *qx = (T *)a.work, *ox = (T *)((char *)a.work + up256((size_t)T_ * a.H * l.kds * sizeof(T)));
    const bool fused = !expand && dtype == AB2_BF16 && a.rank % 8 == 0 && a.dim % 8 == 0 && a.dim <= 256 && a.rot % 8 == 0 && a.stride % 8 == 0;
    cudaError_t e;
    if (!fused) e = launch_kernel(latent_prep_kernel<T>, dim3(a.S, nrows), dim3(256), 0, s, a, expand ? (T *)nullptr : qx);
    else if (a.dim <= 32) e = launch_absorb<1>(a, (__nv_bfloat16 *)qx, T_, s);
    else if (a.dim <= 64) e = launch_absorb<2>(a, (__nv_bfloat16 *)qx, T_, s);
    else if (a.dim <= 128) e = launch_absorb<4>(a, (__nv_bfloat16 *)qx, T_, s);
    else e = launch_absorb<8>(a, (__nv_bfloat16 *)qx, T_, s);
    if (e != cudaSuccess) return fail(AB2_ERR_CUDA, "latent preparation launch failed: %s", cudaGetErrorString(e));
    LinArgs lin = {};
    lin.M = T_; lin.batch = a.H;
    if (!expand) {
        lin.w = a.absorb; lin.wb = (long long)a.rank * a.dim; lin.N = a.rank; lin.K = a.dim;
        lin.x = a.proj; lin.ldx = a.stride; lin.xb = D;
        lin.y = qx; lin.ldy = (long long)a.H * l.kds; lin.yb = l.kds; lin.epi = LIN_STORE;
        int rc = fused ? (int)AB2_OK : linear_dense(lin, dtype, s);
        if (rc == AB2_OK) rc = latent_space_attention<T>(kv, a, qx, ox, nrows, max_len, s);
        if (rc != AB2_OK) return rc;
        lin.w = a.ukv + (size_t)a.dim * a.rank; lin.wb = (long long)(a.dim + a.vdim) * a.rank; lin.N = a.vdim; lin.K = a.rank;
        lin.x = ox; lin.ldx = (long long)a.H * a.rank; lin.xb = a.rank;
        lin.y = a.out; lin.ldy = (long long)a.H * a.vdim; lin.yb = a.vdim;
        if (gate) { lin.epi = LIN_GATE; lin.gate = gate; lin.gate_ld = a.stride; }
        return linear_dense(lin, dtype, s);
    }
    const int heads_at_once = (int)std::min<size_t>(a.H, a.work_bytes / head_bytes);
    for (int r = 0; r < nrows; ++r) {
        const int row = kv_row_host(kv, a.row0, r), first = kv->lens_host[row];
        const __nv_bfloat16 *cached = (const __nv_bfloat16 *)l.k + (size_t)row * l.cap * l.kds;
        const __nv_bfloat16 *proj = (const __nv_bfloat16 *)a.proj + (size_t)r * a.S * a.stride;
        for (int h0 = 0; h0 < a.H; h0 += heads_at_once) {
            const int hn = std::min(heads_at_once, a.H - h0);
            lin.w = a.ukv + (size_t)h0 * (a.dim + a.vdim) * a.rank; lin.N = hn * (a.dim + a.vdim); lin.K = a.rank; lin.M = first + a.S; lin.batch = 1;
            lin.x = cached; lin.ldx = l.kds; lin.y = a.work; lin.ldy = lin.N; lin.epi = LIN_STORE;
            int rc = linear_dense(lin, dtype, s);
            PromptAttnArgs p = {};
            p.q = proj + (size_t)h0 * D; p.q_stride = a.stride; p.k = (const __nv_bfloat16 *)a.work; p.k_stride = lin.N; p.k_head = a.dim + a.vdim;
            p.tail = cached + a.rank; p.tail_stride = l.kds; p.v = p.k + a.dim; p.v_stride = lin.N; p.v_head = p.k_head;
            if (gate) { p.gate = (const __nv_bfloat16 *)gate + (size_t)r * a.S * a.stride + h0; p.gate_stride = a.stride; }
            p.out = (__nv_bfloat16 *)a.out + ((size_t)r * a.S * a.H + h0) * a.vdim; p.out_stride = (long long)a.H * a.vdim;
            p.S = a.S; p.heads = hn; p.first = first; p.dim = a.dim; p.tail_dims = a.rot; p.vdim = a.vdim; p.scale = a.scale;
            if (rc == AB2_OK) rc = prompt_attention(p, s);
            if (rc != AB2_OK) return rc;
        }
    }
    return AB2_OK;
}

}  // namespace

int latent_absorb_weights(const __nv_bfloat16 *ukv, __nv_bfloat16 *absorb, int H, int dim, int vdim, int rank, cudaStream_t s) {
    absorb_weights_kernel<<<dim3((rank + 31) / 32, (dim + 31) / 32, H), dim3(32, 8), 0, s>>>(ukv, absorb, dim, vdim, rank);
    AB2_LAUNCH_CHECK();
    return AB2_OK;
}

// Queries in the latent space and their summed latents, or (a long portion) keys and values of as many
// heads as 256 MB hold, of one at least.
size_t latent_workspace(int H, int dim, int rot, int rank, int vdim, int tokens, int positions, ab2_dtype dtype) {
    const size_t esz = dtype_size(dtype), head = (size_t)positions * (dim + vdim) * 2;
    size_t n = up256((size_t)tokens * H * row_stride(rank, rot) * esz) + up256((size_t)tokens * H * rank * esz);
    if (expandable(dim, rot, rank, vdim, dtype)) n = std::max(n, std::max(head, std::min(head * H, (size_t)256 << 20)));
    return n;
}

int latent_attention(const ab2_kv *kv, LatentArgs a, int nrows, int max_len, ab2_dtype dtype, cudaStream_t s) {
    a.part_acc = kv->part_acc; a.part_ml = kv->part_ml;
    return dtype == AB2_F32 ? launch_latent<float>(kv, a, nrows, max_len, dtype, s) : launch_latent<__nv_bfloat16>(kv, a, nrows, max_len, dtype, s);
}

}  // namespace ab2
