// Mixture-of-experts routing: router scores, group-limited top-k, grouping of the (token, choice) pairs by expert
// and the gather of their rows.  The expert products are in gemm_grouped_sm100.cu (bf16) and gemm_f32.cu, the weighted
// sum of the experts' outputs is part of the norm kernel in block.cu.  Compiled without fast-math.
#include "vec.cuh"

namespace {

// logits[n, e] = h[n, :] . w[e, :], one warp per product; for few tokens (decode)
template <typename T>
__global__ void __launch_bounds__(256)
router_dot_kernel(const T* __restrict__ h, const T* __restrict__ w, float* __restrict__ logits, int E, int D) {
    kb_dep_trigger();
    kb_dep_wait();
    const int e = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (e >= E) return;
    const T* a = h + (long long)blockIdx.x * D;
    const T* b = w + (long long)e * D;
    float acc = 0.f;
    for (int c = lane * 8; c < D; c += 256) {
        float x[8], y[8];
        load8(a + c, x);
        load8(b + c, y);
#pragma unroll
        for (int j = 0; j < 8; ++j) acc += x[j] * y[j];
    }
    acc = warp_sum(acc);
    if (lane == 0) logits[(long long)blockIdx.x * E + e] = acc;
}

// Largest value of v (ties: smallest index) over the warp; returns the index, all lanes agree.
__device__ __forceinline__ int warp_argmax(float& v, int idx) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, v, o);
        const int oi = __shfl_xor_sync(0xffffffffu, idx, o);
        if (ov > v || (ov == v && oi < idx)) { v = ov; idx = oi; }
    }
    return idx;
}

constexpr int SEL_WARPS = 4;
// One warp per token.  Shared memory per warp: E scores and `groups` group scores.
__global__ void __launch_bounds__(SEL_WARPS * 32)
moe_select_kernel(const float* __restrict__ logits, int ld, int N, int E, int top, float scale, int groups, int keep, int gated,
                  int* __restrict__ ids, float* __restrict__ wts, float* __restrict__ gate) {
    extern __shared__ float sel_smem[];
    kb_dep_trigger();
    kb_dep_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int n = blockIdx.x * SEL_WARPS + warp;
    if (n >= N) return;
    float* s = sel_smem + warp * (E + groups);
    float* gs = s + E;
    const float* z = logits + (long long)n * ld;
    float m = -INFINITY;
    for (int e = lane; e < E; e += 32) m = fmaxf(m, z[e]);
    m = warp_max(m);
    float sum = 0.f;
    for (int e = lane; e < E; e += 32) {
        const float p = expf(z[e] - m);
        s[e] = p;
        sum += p;
    }
    sum = warp_sum(sum);
    __syncwarp();
    for (int e = lane; e < E; e += 32) s[e] = s[e] / sum;
    __syncwarp();
    if (keep < groups) {
        const int size = E / groups;
        for (int g = lane; g < groups; g += 32) {
            float b = -INFINITY;
            for (int e = g * size; e < (g + 1) * size; ++e) b = fmaxf(b, s[e]);
            gs[g] = b;
        }
        __syncwarp();
        for (int k = 0; k < keep; ++k) {               // a kept group's score becomes +inf
            float b = -INFINITY;
            int bi = 0x7fffffff;
            for (int g = lane; g < groups; g += 32)
                if (gs[g] != INFINITY && gs[g] > b) { b = gs[g]; bi = g; }
            bi = warp_argmax(b, bi);
            __syncwarp();
            if (lane == 0 && bi < groups) gs[bi] = INFINITY;
            __syncwarp();
        }
        for (int e = lane; e < E; e += 32)
            if (gs[e / size] != INFINITY) s[e] = -1.f;
        __syncwarp();
    }
    for (int k = 0; k < top; ++k) {
        float b = -INFINITY;
        int bi = 0x7fffffff;
        for (int e = lane; e < E; e += 32)
            if (s[e] > b) { b = s[e]; bi = e; }
        bi = warp_argmax(b, bi);
        if (bi >= E) bi = 0;                           // only with non-finite scores
        __syncwarp();
        if (lane == 0) {
            ids[(long long)n * top + k] = bi;
            wts[(long long)n * top + k] = b * scale;
            s[bi] = -2.f;
        }
        __syncwarp();
    }
    if (gated && lane == 0) gate[n] = 1.0f / (1.0f + expf(-z[E]));
}

// Groups the A = N * top choices by expert: at[i] = row of choice i, tok[row] = its token, offsets[E + 1].
// One block; counts and cursors live in shared memory.
constexpr int IDX_THREADS = 1024, IDX_UNROLL = 8, MAX_EXPERTS = 1024;
__global__ void __launch_bounds__(IDX_THREADS)
moe_index_kernel(const int* __restrict__ ids, int A, int top, int E, int* __restrict__ at, int* __restrict__ tok,
                 int* __restrict__ offsets) {
    __shared__ int cnt[MAX_EXPERTS], off[MAX_EXPERTS];
    kb_dep_trigger();
    kb_dep_wait();
    for (int e = threadIdx.x; e < E; e += IDX_THREADS) cnt[e] = 0;
    __syncthreads();
    for (int i0 = threadIdx.x; i0 < A; i0 += IDX_THREADS * IDX_UNROLL) {
        int e[IDX_UNROLL];
#pragma unroll
        for (int u = 0; u < IDX_UNROLL; ++u) {
            const int i = i0 + u * IDX_THREADS;
            e[u] = i < A ? ids[i] : -1;
        }
#pragma unroll
        for (int u = 0; u < IDX_UNROLL; ++u)
            if (e[u] >= 0) at[i0 + u * IDX_THREADS] = atomicAdd(&cnt[e[u]], 1);
    }
    __syncthreads();
    // exclusive prefix sum over the experts (E <= 1024 = block size)
    if (threadIdx.x < MAX_EXPERTS) off[threadIdx.x] = threadIdx.x < (unsigned)E ? cnt[threadIdx.x] : 0;
    __syncthreads();
    for (int d = 1; d < E; d <<= 1) {
        const int v = (int)threadIdx.x >= d ? off[threadIdx.x - d] : 0;
        __syncthreads();
        off[threadIdx.x] += v;
        __syncthreads();
    }
    if (threadIdx.x < (unsigned)E) offsets[threadIdx.x + 1] = off[threadIdx.x];
    if (threadIdx.x == 0) offsets[0] = 0;
    for (int i0 = threadIdx.x; i0 < A; i0 += IDX_THREADS * IDX_UNROLL) {
        int e[IDX_UNROLL], r[IDX_UNROLL];
#pragma unroll
        for (int u = 0; u < IDX_UNROLL; ++u) {
            const int i = i0 + u * IDX_THREADS;
            e[u] = i < A ? ids[i] : -1;
            r[u] = i < A ? at[i] : 0;
        }
#pragma unroll
        for (int u = 0; u < IDX_UNROLL; ++u)
            if (e[u] >= 0) {
                const int i = i0 + u * IDX_THREADS;
                const int row = off[e[u]] - cnt[e[u]] + r[u];
                at[i] = row;
                tok[row] = i / top;
            }
    }
}

// out[r] = h[tok[r]], 16 bytes per thread and step
__global__ void moe_gather_kernel(const uint4* __restrict__ h, const int* __restrict__ tok, uint4* __restrict__ out, int A, int vecs) {
    kb_dep_trigger();
    kb_dep_wait();
    const long long total = (long long)A * vecs;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
        const int r = (int)(i / vecs), c = (int)(i % vecs);
        out[i] = h[(long long)tok[r] * vecs + c];
    }
}

}  // namespace

KB_API int kb_router_dot(const void* h, const void* w, float* logits, int N, int E, int D, int type, cudaStream_t st) {
    if (D % 8 || N < 1 || E < 1) return 5;
    const dim3 grid(N, (E + 7) / 8);
    if (type == 0) return kb_launch_dep(router_dot_kernel<bf16>, grid, dim3(256), 0, st, (const bf16*)h, (const bf16*)w, logits, E, D);
    return kb_launch_dep(router_dot_kernel<float>, grid, dim3(256), 0, st, (const float*)h, (const float*)w, logits, E, D);
}
// logits[N, ld]: E expert logits per token and, with `gated`, the gate's logit behind them.
KB_API int kb_moe_select(const float* logits, int ld, int N, int E, int top, float scale, int groups, int keep, int gated, int* ids,
                         float* wts, float* gate, cudaStream_t st) {
    if (N < 1 || E < 1 || E > MAX_EXPERTS || groups < 1 || E % groups || keep < 1 || keep > groups || top < 1 ||
        top > keep * (E / groups) || ld < E + (gated ? 1 : 0))
        return 5;
    return kb_launch_dep(moe_select_kernel, dim3((N + SEL_WARPS - 1) / SEL_WARPS), dim3(SEL_WARPS * 32),
                         (size_t)SEL_WARPS * (E + groups) * 4, st, logits, ld, N, E, top, scale, groups, keep, gated, ids, wts, gate);
}
// at / tok: [N * top]; offsets: [E + 1]; rows: gathered copies of h's rows, [N * top, row_bytes]
KB_API int kb_moe_group(const void* h, const int* ids, int N, int top, int E, int row_bytes, int* at, int* tok, int* offsets,
                        void* rows, cudaStream_t st) {
    const long long A = (long long)N * top;
    if (N < 1 || top < 1 || E < 1 || E > MAX_EXPERTS || row_bytes % 16 || A > 0x7fffffff) return 5;
    const int r = kb_launch_dep(moe_index_kernel, dim3(1), dim3(IDX_THREADS), 0, st, ids, (int)A, top, E, at, tok, offsets);
    if (r) return r;
    long long blocks = (A * (row_bytes / 16) + 255) / 256;
    if (blocks > 148 * 16) blocks = 148 * 16;
    return kb_launch_dep(moe_gather_kernel, dim3((unsigned)blocks), dim3(256), 0, st, (const uint4*)h, (const int*)tok, (uint4*)rows,
                         (int)A, row_bytes / 16);
}
