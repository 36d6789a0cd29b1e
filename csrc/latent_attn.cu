// Attention over cached latents in its plain form, for the 32-bit mode and for sizes the tensor-core kernel does not
// take: every head scores its latent-space query against the cached rows and averages the same rows.  One block per
// (token, head), an online softmax over tiles of 128 rows.  Compiled without fast-math.
#include "vec.cuh"

namespace {

constexpr int PAGE = 16, TILE = 128, MAXE = 8;         // latent sizes up to TILE * MAXE

template <typename T>
__global__ void __launch_bounds__(TILE)
latent_attn_kernel(const T* __restrict__ q, const T* __restrict__ pages, int W, const int* __restrict__ table, int max_pages, int num_pages,
                   const int* __restrict__ ctx_lens, const int* __restrict__ cu, int B, T* __restrict__ out, int H, int R, float scale,
                   int* __restrict__ status) {
    extern __shared__ float la_smem[];
    float* qs = la_smem;                               // [R]
    float* ps = qs + R;                                // [TILE]
    const T** rowp = reinterpret_cast<const T**>(ps + TILE);   // [TILE] cache row of every key of the tile
    __shared__ float red[2][TILE / 32];
    kb_dep_trigger();
    kb_dep_wait();
    const int n = blockIdx.x, head = blockIdx.y, t = threadIdx.x, lane = t & 31, warp = t >> 5;
    int b = n, last = 0;                               // sequence, and how many of its tokens follow this one in the pass
    if (cu) {
        int lo = 0, hi = B;
        while (hi - lo > 1) {
            const int m = (lo + hi) >> 1;
            if (cu[m] <= n) lo = m; else hi = m;
        }
        b = lo;
        last = cu[b + 1] - 1 - n;
    }
    const int keys = min(ctx_lens[b] - last, max_pages * PAGE);
    const T* qrow = q + ((long long)n * H + head) * R;
    for (int i = t; i < R; i += TILE) qs[i] = to_float(qrow[i]);
    float o[MAXE];
#pragma unroll
    for (int i = 0; i < MAXE; ++i) o[i] = 0.f;
    float m = -INFINITY, l = 0.f;
    for (int k0 = 0; k0 < keys; k0 += TILE) {
        const int k = k0 + t;
        const T* row = nullptr;
        if (k < keys) {
            const int page = table[(long long)b * max_pages + k / PAGE];
            if (page >= 0 && page < num_pages) row = pages + (long long)page * PAGE * R + (k % PAGE) * W;
            else if (status) atomicMax(status, (int)KB_BAD_INDEX);
        }
        __syncthreads();                               // qs is there; the previous tile's ps and rowp are done with
        rowp[t] = row;
        float s = -INFINITY;
        if (row) {
            s = 0.f;
            for (int i = 0; i < R; i += 8) {
                float c[8];
                load8(row + (i / W) * PAGE * W + i % W, c);
#pragma unroll
                for (int j = 0; j < 8; ++j) s = fmaf(qs[i + j], c[j], s);
            }
            s *= scale;
        }
        const float wm = warp_max(s);
        if (lane == 0) red[0][warp] = wm;
        __syncthreads();
        float mn = m;
#pragma unroll
        for (int w = 0; w < TILE / 32; ++w) mn = fmaxf(mn, red[0][w]);
        const float p = row ? expf(s - mn) : 0.f;
        ps[t] = p;
        const float wsum = warp_sum(p);
        if (lane == 0) red[1][warp] = wsum;
        __syncthreads();
        const float f = m == -INFINITY ? 0.f : expf(m - mn);
        m = mn;
        l = l * f;
#pragma unroll
        for (int w = 0; w < TILE / 32; ++w) l += red[1][w];
        const int nk = min(TILE, keys - k0);
#pragma unroll
        for (int i = 0; i < MAXE; ++i) {
            const int r = i * TILE + t;
            if (r >= R) break;
            const int at = (r / W) * PAGE * W + r % W;
            float a = o[i] * f;
            for (int j = 0; j < nk; ++j)
                if (rowp[j]) a = fmaf(ps[j], to_float(rowp[j][at]), a);
            o[i] = a;
        }
    }
    T* dst = out + ((long long)n * H + head) * R;
#pragma unroll
    for (int i = 0; i < MAXE; ++i) {
        const int r = i * TILE + t;
        if (r < R) from_float(dst + r, l > 0.f ? o[i] / l : 0.f);
    }
}

}  // namespace

// q, out: [N, H, R]; pages: [num_pages, R / W, 16, W]; cu null: row n is sequence n.
KB_API int kb_latent_attn_plain(const void* q, const void* pages, int W, const int* table, int max_pages, int num_pages, const int* ctx_lens,
                                const int* cu, int B, void* out, int N, int H, int R, float scale, int type, int* status,
                                cudaStream_t st) {
    if (N < 1 || H < 1 || B < 1 || R % 8 || R > TILE * MAXE || W < 8 || W % 8 || R % W) return 5;
    const size_t smem = (size_t)(R + TILE) * 4 + TILE * sizeof(void*);
    if (type == 0)
        return kb_launch_dep(latent_attn_kernel<bf16>, dim3(N, H), dim3(TILE), smem, st, (const bf16*)q, (const bf16*)pages, W, table,
                             max_pages, num_pages, ctx_lens, cu, B, (bf16*)out, H, R, scale, status);
    return kb_launch_dep(latent_attn_kernel<float>, dim3(N, H), dim3(TILE), smem, st, (const float*)q, (const float*)pages, W, table,
                         max_pages, num_pages, ctx_lens, cu, B, (float*)out, H, R, scale, status);
}
