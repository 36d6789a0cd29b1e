// Mixture-of-experts routing: router scores, group-limited top-k, grouping of the (token, choice) pairs by expert
// and the gather of their rows.  Few tokens (decoding): one kernel scores and selects, one groups and gathers, each
// block finding its places in the grouping from all the choices.  Many tokens: the scores are a matrix product, the
// selection counts the experts' choices with atomics, the gather turns the counts into places.  The order of an
// expert's rows does not matter: rows are independent, and a token's outputs are summed in the order of its choices.
// The expert products are in gemm_grouped_sm100.cu (bf16) and gemm_f32.cu, the weighted sum of the experts' outputs
// is part of the norm kernel in block.cu.  Compiled without fast-math.
#include "vec.cuh"

namespace {

constexpr int MAX_EXPERTS = 1024;

struct Select {
    int E, top, groups, keep, gated;
    float scale;
    int* ids;                      // [N, top]
    float* wts;                    // [N, top]
    float* gate;                   // [N]
    int* counts;                   // [E] choices per expert, null: not counted
    int* rank;                     // [N, top] place of the choice among its expert's
};

// Index of the largest value over the warp (ties: smallest index); every lane brings its best (key 0: none).  Keys are
// the bits of non-negative floats plus one, which compare like the floats.
__device__ __forceinline__ int warp_argmax(uint32_t key, int idx) {
    const uint32_t m = __reduce_max_sync(0xffffffffu, key);
    return (int)__reduce_min_sync(0xffffffffu, key == m && m != 0u ? (uint32_t)idx : 0x7fffffffu);
}

// One warp selects for token n; z: E logits (and the gate's behind them); s: E + groups floats of shared memory.
__device__ __forceinline__ void select_experts(const float* z, float* s, const Select& c, int n, int lane) {
    float* gs = s + c.E;
    float m = -INFINITY;
    for (int e = lane; e < c.E; e += 32) m = fmaxf(m, z[e]);
    m = warp_max(m);
    float sum = 0.f;
    for (int e = lane; e < c.E; e += 32) {
        const float p = expf(z[e] - m);
        s[e] = p;
        sum += p;
    }
    sum = warp_sum(sum);
    __syncwarp();
    const int size = c.E / c.groups;
    const bool limited = c.keep < c.groups;
    if (limited) {
        for (int g = lane; g < c.groups; g += 32) {
            float b = 0.f;
            for (int e = g * size; e < (g + 1) * size; ++e) b = fmaxf(b, s[e]);
            gs[g] = b;
        }
        __syncwarp();
        for (int k = 0; k < c.keep; ++k) {             // a kept group's score becomes -1
            uint32_t b = 0u;
            int bi = 0x7fffffff;
            for (int g = lane; g < c.groups; g += 32)
                if (gs[g] >= 0.f && __float_as_uint(gs[g]) + 1u > b) { b = __float_as_uint(gs[g]) + 1u; bi = g; }
            bi = warp_argmax(b, bi);
            if (lane == 0 && bi < c.groups) gs[bi] = -1.f;
            __syncwarp();
        }
        for (int e = lane; e < c.E; e += 32)
            if (gs[e / size] >= 0.f) s[e] = -1.f;
        __syncwarp();
    }
    for (int k = 0; k < c.top; ++k) {
        uint32_t b = 0u;
        int bi = 0x7fffffff;
        for (int e = lane; e < c.E; e += 32)
            if (s[e] >= 0.f && __float_as_uint(s[e]) + 1u > b) { b = __float_as_uint(s[e]) + 1u; bi = e; }
        bi = warp_argmax(b, bi);
        if (bi >= c.E) bi = 0;                         // only with non-finite scores
        __syncwarp();
        if (lane == 0) {
            const long long i = (long long)n * c.top + k;
            c.ids[i] = bi;
            c.wts[i] = s[bi] / sum * c.scale;
            if (c.counts) c.rank[i] = atomicAdd(&c.counts[bi], 1);
            s[bi] = -1.f;
        }
        __syncwarp();
    }
    if (c.gated && lane == 0) c.gate[n] = 1.0f / (1.0f + expf(-z[c.E]));
}

// Few tokens: one block per token, a warp per expert at a time, then the first warp selects.
template <typename T>
__global__ void __launch_bounds__(512)
route_token_kernel(const T* __restrict__ h, const T* __restrict__ w, int rows, int D, const Select c) {
    extern __shared__ float rt_smem[];
    float* x = rt_smem;                                // [D]
    float* z = x + D;                                  // [rows]
    kb_dep_trigger();
    kb_dep_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    for (int i = threadIdx.x * 8; i < D; i += 512 * 8) load8(h + (long long)blockIdx.x * D + i, x + i);
    __syncthreads();
    for (int e = warp; e < rows; e += 16) {
        const T* b = w + (long long)e * D;
        float acc = 0.f;
#pragma unroll 4
        for (int i = lane * 8; i < D; i += 256) {
            float y[8];
            load8(b + i, y);
#pragma unroll
            for (int j = 0; j < 8; ++j) acc += x[i + j] * y[j];
        }
        acc = warp_sum(acc);
        if (lane == 0) z[e] = acc;
    }
    __syncthreads();
    if (warp == 0) select_experts(z, z + rows, c, blockIdx.x, lane);
}

// Many tokens: one warp per token on the logits of a matrix product.
constexpr int SEL_WARPS = 4;
__global__ void __launch_bounds__(SEL_WARPS * 32)
moe_select_kernel(const float* __restrict__ logits, int ld, int N, const Select c) {
    extern __shared__ float sel_smem[];
    kb_dep_trigger();
    kb_dep_wait();
    const int warp = threadIdx.x >> 5, n = blockIdx.x * SEL_WARPS + warp;
    if (n < N) select_experts(logits + (long long)n * ld, sel_smem + warp * (c.E + c.groups), c, n, threadIdx.x & 31);
}

// One block per token: the places at[n, k] of its choices in the grouping, offsets[E + 1], and copies of the token's row
// to these places.  FEW: counts and ranks are found here from all choices (`A` of them); otherwise the selection has left
// them in `counts` and `at`.
template <bool FEW>
__global__ void __launch_bounds__(256)
moe_gather_kernel(const uint4* __restrict__ h, const int* __restrict__ ids, const int* __restrict__ counts, int* __restrict__ at,
                  int* __restrict__ offsets, uint4* __restrict__ out, int A, int top, int E, int vecs, int* __restrict__ status) {
    extern __shared__ int mg_smem[];
    int* off = mg_smem;                                // [E] counts, then exclusive prefix sums
    int* place = off + E;                              // [top]
    __shared__ int wsum[8];
    kb_dep_trigger();
    kb_dep_wait();
    const int n = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    for (int e = threadIdx.x; e < E; e += 256) off[e] = FEW ? 0 : counts[e];
    for (int k = threadIdx.x; k < top; k += 256) place[k] = FEW ? 0 : at[(long long)n * top + k];
    __syncthreads();
    if (FEW) {
        for (int i = threadIdx.x; i < A; i += 256) {
            const int e = ids[i];
            atomicAdd(&off[e], 1);
            // choices in front of this token's, and its own earlier ones (a token's choices differ)
            if (i < n * top)
                for (int k = 0; k < top; ++k)
                    if (ids[n * top + k] == e) atomicAdd(&place[k], 1);
        }
        __syncthreads();
    }
    // exclusive prefix sums: a run of experts per thread
    const int per = (E + 255) / 256;
    int mine = 0;
    for (int i = 0; i < per; ++i) {
        const int e = threadIdx.x * per + i;
        if (e < E) mine += off[e];
    }
    int s = mine;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const int v = __shfl_up_sync(0xffffffffu, s, o);
        if (lane >= o) s += v;
    }
    if (lane == 31) wsum[warp] = s;
    __syncthreads();
    int run = s - mine;
    for (int v = 0; v < warp; ++v) run += wsum[v];
    for (int i = 0; i < per; ++i) {
        const int e = threadIdx.x * per + i;
        if (e < E) {
            const int cnt = off[e];
            off[e] = run;
            run += cnt;
            if (n == 0) offsets[e + 1] = run;
        }
    }
    if (n == 0 && threadIdx.x == 0) offsets[0] = 0;
    __syncthreads();
    for (int k = threadIdx.x; k < top; k += 256) {
        int row = off[ids[(long long)n * top + k]] + place[k];
        if (row < 0 || row >= A) {
            if (status) atomicMax(status, (int)KB_BAD_INDEX);
            row = -1;
        }
        place[k] = row;
        at[(long long)n * top + k] = row;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < vecs; i += 256) {
        const uint4 v = h[(long long)n * vecs + i];
        for (int k = 0; k < top; ++k)
            if (place[k] >= 0) out[(long long)place[k] * vecs + i] = v;
    }
}

inline bool select_ok(int N, const Select& c) {
    return N >= 1 && c.E >= 1 && c.E <= MAX_EXPERTS && c.groups >= 1 && c.E % c.groups == 0 && c.keep >= 1 && c.keep <= c.groups &&
           c.top >= 1 && c.top <= c.keep * (c.E / c.groups);
}

}  // namespace

// Router and selection for few tokens.  w: [E (+ 1 with `gated`), D]; ids, wts: [N, top]; gate: [N] or null.
KB_API int kb_moe_route_few(const void* h, const void* w, int N, int E, int D, int top, float scale, int groups, int keep, int gated,
                            int* ids, float* wts, float* gate, int type, cudaStream_t st) {
    const Select c{E, top, groups, keep, gated, scale, ids, wts, gate, nullptr, nullptr};
    const int rows = E + (gated ? 1 : 0);
    const size_t smem = (size_t)(D + rows + E + groups) * 4;
    if (D % 8 || !select_ok(N, c) || smem > 48 * 1024) return 5;
    if (type == 0)
        return kb_launch_dep(route_token_kernel<bf16>, dim3(N), dim3(512), smem, st, (const bf16*)h, (const bf16*)w, rows, D, c);
    return kb_launch_dep(route_token_kernel<float>, dim3(N), dim3(512), smem, st, (const float*)h, (const float*)w, rows, D, c);
}
// Selection on logits[N, ld] (E expert logits and, with `gated`, the gate's).  counts[E] (zero) and rank[N, top] receive
// what kb_moe_group needs.
KB_API int kb_moe_select(const float* logits, int ld, int N, int E, int top, float scale, int groups, int keep, int gated, int* ids,
                         float* wts, float* gate, int* counts, int* rank, cudaStream_t st) {
    const Select c{E, top, groups, keep, gated, scale, ids, wts, gate, counts, rank};
    if (!select_ok(N, c) || ld < E + (gated ? 1 : 0)) return 5;
    return kb_launch_dep(moe_select_kernel, dim3((N + SEL_WARPS - 1) / SEL_WARPS), dim3(SEL_WARPS * 32),
                         (size_t)SEL_WARPS * (E + groups) * 4, st, logits, ld, N, c);
}
// Groups the N * top choices by expert: at[N, top] (with counts: holds the ranks on entry), offsets[E + 1], rows
// [N * top, row_bytes] = copies of h's rows.  counts null: everything is found from ids (few tokens).
KB_API int kb_moe_group(const void* h, const int* ids, const int* counts, int N, int top, int E, int row_bytes, int* at, int* offsets,
                        void* rows, int* status, cudaStream_t st) {
    const long long A = (long long)N * top;
    if (N < 1 || top < 1 || E < 1 || E > MAX_EXPERTS || top > E || row_bytes % 16 || A > 0x7fffffff) return 5;
    const size_t smem = (size_t)(E + top) * 4;
    if (counts)
        return kb_launch_dep(moe_gather_kernel<false>, dim3(N), dim3(256), smem, st, (const uint4*)h, ids, counts, at, offsets,
                             (uint4*)rows, (int)A, top, E, row_bytes / 16, status);
    return kb_launch_dep(moe_gather_kernel<true>, dim3(N), dim3(256), smem, st, (const uint4*)h, ids, counts, at, offsets, (uint4*)rows,
                         (int)A, top, E, row_bytes / 16, status);
}
