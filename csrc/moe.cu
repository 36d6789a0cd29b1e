// Mixture-of-experts routing: router scores, group-limited top-k, grouping of the (token, choice) pairs by expert
// and the gather of their rows.  Few tokens (decoding): the scores are dot products, and each block of the gather finds
// its places in the grouping from all the choices.  Many tokens: the scores are a matrix product, the selection
// counts the experts' choices with atomics, the gather turns the counts into places.  The order of an
// expert's rows does not matter: rows are independent, and a token's outputs are summed in the order of its choices.
// The expert products are in gemm_grouped_sm100.cu (bf16) and gemm_f32.cu, the weighted sum of the experts' outputs
// is part of the norm kernel in block.cu.  Compiled without fast-math.
#include "vec.cuh"

namespace {

constexpr int MAX_EXPERTS = 1024;
constexpr int COUNT_STRIDE = 32;   // ints between the experts' counters: one cache line each, or the atomics queue up

struct Select {
    int E, top, groups, keep, gated;
    float scale;
    int* ids;                      // [N, top]
    float* wts;                    // [N, top]
    float* gate;                   // [N]
    int* counts;                   // [E * COUNT_STRIDE] choices per expert, null: not counted
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
    const float norm = c.scale / sum;
    for (int k0 = 0; k0 < c.top; k0 += 32) {           // lane k keeps choice k: stores and atomics of 32 choices go together
        const int n_k = min(32, c.top - k0);
        int mine = 0;
        float score = 0.f;
        for (int k = 0; k < n_k; ++k) {
            uint32_t b = 0u;
            int bi = 0x7fffffff;
            for (int e = lane; e < c.E; e += 32)
                if (s[e] >= 0.f && __float_as_uint(s[e]) + 1u > b) { b = __float_as_uint(s[e]) + 1u; bi = e; }
            bi = warp_argmax(b, bi);
            if (bi >= c.E) bi = 0;                     // only with non-finite scores
            if (lane == k) {
                mine = bi;
                score = s[bi];
            }
            __syncwarp();
            if (lane == 0) s[bi] = -1.f;
            __syncwarp();
        }
        if (lane < n_k) {
            const long long i = (long long)n * c.top + k0 + lane;
            c.ids[i] = mine;
            c.wts[i] = score * norm;
            if (c.counts) c.rank[i] = atomicAdd(&c.counts[mine * COUNT_STRIDE], 1);
        }
    }
    if (c.gated && lane == 0) c.gate[n] = 1.0f / (1.0f + expf(-z[c.E]));
}

// Few tokens: logits[n, e] = h[n, :] . w[e, :].  A block takes eight tokens (their rows in shared memory) and eight
// experts, one per warp, so that a row of w is read once for eight tokens.
constexpr int DOT_TOKENS = 8;
template <typename T>
__global__ void __launch_bounds__(256)
router_dot_kernel(const T* __restrict__ h, const T* __restrict__ w, float* __restrict__ logits, int N, int E, int D) {
    extern __shared__ __align__(16) uint8_t rd_smem[];
    T* x = reinterpret_cast<T*>(rd_smem);              // [DOT_TOKENS][D]
    kb_dep_trigger();
    const int n0 = blockIdx.x * DOT_TOKENS, e = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    kb_dep_wait();
    constexpr int V = 16 / sizeof(T);
    for (int i = threadIdx.x; i < DOT_TOKENS * D / V; i += 256) {
        const int t = min(n0 + i / (D / V), N - 1);
        reinterpret_cast<uint4*>(x)[i] = reinterpret_cast<const uint4*>(h + (long long)t * D)[i % (D / V)];
    }
    __syncthreads();
    if (e >= E) return;
    const T* b = w + (long long)e * D;
    float acc[DOT_TOKENS] = {};
#pragma unroll 4
    for (int i = lane * 8; i < D; i += 256) {
        float y[8];
        load8(b + i, y);
#pragma unroll
        for (int t = 0; t < DOT_TOKENS; ++t) {
            float v[8];
            load8(x + t * D + i, v);
#pragma unroll
            for (int j = 0; j < 8; ++j) acc[t] += v[j] * y[j];
        }
    }
#pragma unroll
    for (int t = 0; t < DOT_TOKENS; ++t) {
        acc[t] = warp_sum(acc[t]);
        if (lane == t && n0 + t < N) logits[(long long)(n0 + t) * E + e] = acc[t];
    }
}

// One warp per token.
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
    for (int e = threadIdx.x; e < E; e += 256) off[e] = FEW ? 0 : counts[e * COUNT_STRIDE];
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

// logits[N, E] for few tokens (their rows are staged in shared memory, eight at a time).
KB_API int kb_router_dot(const void* h, const void* w, float* logits, int N, int E, int D, int type, cudaStream_t st) {
    const size_t smem = (size_t)DOT_TOKENS * D * (type == 0 ? 2 : 4);
    if (D % 8 || N < 1 || E < 1 || smem > 200 * 1024) return 5;
    static bool flags[2][64] = {};
    bool* set = kb_device_flag(flags[type == 0 ? 0 : 1]);
    if (!set) return 7;
    if (!*set) {
        if ((type == 0 ? cudaFuncSetAttribute(router_dot_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024)
                       : cudaFuncSetAttribute(router_dot_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024)) !=
            cudaSuccess)
            return 7;
        *set = true;
    }
    const dim3 grid((N + DOT_TOKENS - 1) / DOT_TOKENS, (E + 7) / 8);
    if (type == 0) return kb_launch_dep(router_dot_kernel<bf16>, grid, dim3(256), smem, st, (const bf16*)h, (const bf16*)w, logits, N, E, D);
    return kb_launch_dep(router_dot_kernel<float>, grid, dim3(256), smem, st, (const float*)h, (const float*)w, logits, N, E, D);
}
// Selection on logits[N, ld] (E expert logits and, with `gated`, the gate's).  ids, wts: [N, top]; gate: [N] or null.
// counts[32 E] (every 32nd used, zero on entry) and rank[N, top] receive what kb_moe_group needs; null: not wanted.
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
