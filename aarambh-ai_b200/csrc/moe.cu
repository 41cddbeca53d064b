// Routing of a mixture of experts: sigmoid scores of the router's f32 logits and the `top` largest per
// token, or experts named by a table of token ids; and the (token, expert) pairs sorted by expert for the
// grouped linears.
#include <algorithm>
#include <climits>

#include "stack.cuh"

using namespace ab2;

namespace ab2 {
namespace {

constexpr int MAX_EXPERTS = 1024;
constexpr int ONE_CTA_PAIRS = 4096;  // up to here one CTA does it all

// The `top` largest of a token's E logits by one warp (the sigmoid keeps the order; equal logits: the
// lower expert first).
__device__ __forceinline__ void choose_experts(const float *z, int E, int top, int *expert, float *score, int lane) {
    // a key that orders like (logit, lower index first); taken ones fall below every logit
    uint32_t taken = 0;  // bit i: this lane's expert lane + 32 i
    for (int k = 0; k < top; ++k) {
        float best = -INFINITY;
        int be = INT_MAX;
        for (int i = 0; lane + 32 * i < E; ++i) {
            const float v = z[lane + 32 * i];
            if (!((taken >> i) & 1u) && (v > best || be == INT_MAX)) { best = v; be = lane + 32 * i; }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, best, o);
            const int oe = __shfl_xor_sync(0xffffffffu, be, o);
            if (oe != INT_MAX && (be == INT_MAX || ov > best || (ov == best && oe < be))) { best = ov; be = oe; }
        }
        if ((be & 31) == lane) taken |= 1u << (be >> 5);
        if (lane == 0) {
            expert[k] = be;
            score[k] = 1.f / (1.f + expf(-best));
        }
    }
}

__global__ void __launch_bounds__(256) moe_choose_kernel(const float *logits, int T, MoeRoute r) {
    pdl_wait();
    pdl_launch_dependents();
    const int t = blockIdx.x * 8 + (threadIdx.x >> 5);
    if (t < T) choose_experts(logits + (size_t)t * r.E, r.E, r.top, r.expert + (size_t)t * r.top, r.score + (size_t)t * r.top, threadIdx.x & 31);
}

// Counting sort of the pairs by expert, by one CTA whose threads have written r.expert.
__device__ __forceinline__ void sort_pairs(const MoeRoute &r, int *count, int *next) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int e = threadIdx.x; e < r.E; e += blockDim.x) count[e] = 0;
    __syncthreads();
    for (int p = threadIdx.x; p < r.pairs; p += blockDim.x) atomicAdd(&count[r.expert[p]], 1);
    __syncthreads();
    if (warp == 0) {
        int base = 0, nact = 0;
        for (int e0 = 0; e0 < r.E; e0 += 32) {
            const int e = e0 + lane, n = e < r.E ? count[e] : 0;
            int inc = n;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int v = __shfl_up_sync(0xffffffffu, inc, o);
                if (lane >= o) inc += v;
            }
            const unsigned live = __ballot_sync(0xffffffffu, n > 0);
            if (e < r.E) { next[e] = base + inc - n; r.offset[e] = base + inc - n; }
            if (n > 0) r.active[1 + nact + __popc(live & ((1u << lane) - 1u))] = e;
            nact += __popc(live);
            base += __shfl_sync(0xffffffffu, inc, 31);
        }
        if (lane == 0) { r.offset[r.E] = base; r.active[0] = nact; }
    }
    __syncthreads();
    for (int p = threadIdx.x; p < r.pairs; p += blockDim.x) r.perm[atomicAdd(&next[r.expert[p]], 1)] = p;
}

// One CTA: (with CHOOSE) the choice, then the sort.
template <bool CHOOSE>
__global__ void __launch_bounds__(1024) moe_sort_kernel(const float *logits, int T, MoeRoute r) {
    __shared__ int count[MAX_EXPERTS], next[MAX_EXPERTS];
    pdl_wait();
    pdl_launch_dependents();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
    if (CHOOSE)
        for (int t = warp; t < T; t += nw)
            choose_experts(logits + (size_t)t * r.E, r.E, r.top, r.expert + (size_t)t * r.top, r.score + (size_t)t * r.top, lane);
    sort_pairs(r, count, next);
}

// One CTA per layer whose experts are named by the token id.
__global__ void __launch_bounds__(1024) moe_table_kernel(const MoeTable *tables, const uint32_t *ids, int vocab, int T) {
    __shared__ int count[MAX_EXPERTS], next[MAX_EXPERTS];
    pdl_wait();
    pdl_launch_dependents();
    const MoeTable m = tables[blockIdx.x];
    MoeRoute r = m.r;
    r.pairs = T * r.top;
    for (int p = threadIdx.x; p < r.pairs; p += blockDim.x) {
        const uint32_t id = min(ids[p / r.top], (uint32_t)vocab - 1u);  // ids are validated on the host; keep reads in range
        r.expert[p] = m.table[(size_t)id * r.top + p % r.top];
    }
    sort_pairs(r, count, next);
}

}  // namespace

int moe_route(const float *logits, int T, const MoeRoute &r, cudaStream_t s) {
    AB2_REQUIRE(r.E <= MAX_EXPERTS, AB2_ERR_UNSUPPORTED, "%d experts exceed the %d the router serves", r.E, MAX_EXPERTS);
    cudaError_t e;
    if (r.pairs <= ONE_CTA_PAIRS && T <= 64) {
        e = launch_kernel(moe_sort_kernel<true>, dim3(1), dim3(T <= 8 ? 256 : 1024), 0, s, logits, T, r);
    } else {
        e = launch_kernel(moe_choose_kernel, dim3((T + 7) / 8), dim3(256), 0, s, logits, T, r);
        if (e == cudaSuccess) e = launch_kernel(moe_sort_kernel<false>, dim3(1), dim3(1024), 0, s, logits, T, r);
    }
    if (e != cudaSuccess) return fail(AB2_ERR_CUDA, "routing launch failed: %s", cudaGetErrorString(e));
    return AB2_OK;
}

int moe_route_tables(const MoeTable *tables_dev, int n, const uint32_t *ids, int vocab, int T, cudaStream_t s) {
    cudaError_t e = launch_kernel(moe_table_kernel, dim3(n), dim3(T <= 8 ? 128 : 1024), 0, s, tables_dev, ids, vocab, T);
    if (e != cudaSuccess) return fail(AB2_ERR_CUDA, "routing launch failed: %s", cudaGetErrorString(e));
    return AB2_OK;
}

}  // namespace ab2
