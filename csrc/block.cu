// Per-token steps of decoders: pair embedding, latent norm + cache append, cache gather, output norm + layer
// scale + residual, residual + pre-norm, final norm, activations, logit soft-cap.
// The residual stream is fp32; T (bf16 or fp32) is the activation type.  Rows may be padded with zeros on the
// right up to a multiple of 8 elements: `width` is the true size that means are taken over.
// Compiled without fast-math: the fp32 mode is meant to be exact to fp32 rounding.
#include "act.cuh"
#include "vec.cuh"

namespace {

constexpr int PAGE = 16;

template <typename T>
__global__ void embed_pairs_kernel(const long long* __restrict__ ids, const int* __restrict__ prev, const T* __restrict__ table,
                                   const T* __restrict__ bigram, long long buckets, long long mul_prev, long long mul_cur,
                                   float scale, float* __restrict__ x, T* __restrict__ h, int N, int D, int V,
                                   int* __restrict__ status) {
    kb_dep_trigger();
    kb_dep_wait();
    const int dc = D >> 3;
    const long long total = (long long)N * dc;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
        const int row = (int)(i / dc), c = (int)(i % dc) * 8;
        const long long id = ids[row];
        float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
        if (id < 0 || id >= V) {
            if (c == 0 && status) atomicMax(status, (int)KB_BAD_INDEX);
        } else {
            load8(table + id * D + c, v);
            if (bigram) {
                const long long p = prev[row];
                const long long b = p < 0 ? buckets : (p * mul_prev + id * mul_cur) % buckets;
                float w[8];
                load8(bigram + b * D + c, w);
#pragma unroll
                for (int j = 0; j < 8; ++j) v[j] += w[j];
            }
#pragma unroll
            for (int j = 0; j < 8; ++j) v[j] *= scale;
        }
        store8(x + (long long)row * D + c, v);
        if (h && (const void*)h != (const void*)x) store8(h + (long long)row * D + c, v);
    }
}

// One warp per row: RMS norm of R elements, to the packed rows and to the row's cache slot.
template <typename T>
__global__ void __launch_bounds__(256)
latent_append_kernel(const T* __restrict__ rows, long long stride, const float* __restrict__ w, int width, float eps,
                     T* __restrict__ pages, int W, const long long* __restrict__ slots, T* __restrict__ out, int N, int R,
                     long long num_slots, int* __restrict__ status) {
    kb_dep_trigger();
    kb_dep_wait();
    const int row = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (row >= N) return;
    const T* src = rows + (long long)row * stride;
    float ss = 0.f;
    for (int c = lane * 8; c < R; c += 256) {
        float v[8];
        load8(src + c, v);
#pragma unroll
        for (int j = 0; j < 8; ++j) ss += v[j] * v[j];
    }
    const float r = 1.0f / sqrtf(warp_sum(ss) / (float)width + eps);
    long long s = slots[row];
    if (s >= num_slots) {
        if (lane == 0 && status) atomicMax(status, (int)KB_BAD_INDEX);
        s = -1;
    }
    for (int c = lane * 8; c < R; c += 256) {
        float v[8], g[8];
        load8(src + c, v);
        load8(w + c, g);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = v[j] * r * g[j];
        if (out) store8(out + (long long)row * R + c, v);
        if (s >= 0) store8(pages + (s / PAGE) * PAGE * R + ((long long)(c / W) * PAGE + s % PAGE) * W + c % W, v);
    }
}

// Packed copy of the cached rows of every sequence; row -> sequence by binary search in the prefix sums.
template <typename T>
__global__ void latent_gather_kernel(const T* __restrict__ pages, int W, const int* __restrict__ table, int max_pages,
                                     const int* __restrict__ cu, int B, T* __restrict__ out, int total, int R, int num_pages,
                                     int* __restrict__ status) {
    kb_dep_trigger();
    kb_dep_wait();
    const int rc = R >> 3;
    const long long n = (long long)total * rc;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
        const int row = (int)(i / rc), c = (int)(i % rc) * 8;
        int lo = 0, hi = B;                            // the sequence b with cu[b] <= row < cu[b + 1]
        while (hi - lo > 1) {
            const int m = (lo + hi) >> 1;
            if (cu[m] <= row) lo = m; else hi = m;
        }
        const int t = row - cu[lo], pi = t / PAGE;
        const int page = pi < max_pages ? table[(long long)lo * max_pages + pi] : -1;
        float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
        if (page < 0 || page >= num_pages) {
            if (c == 0 && status) atomicMax(status, (int)KB_BAD_INDEX);
        } else {
            load8(pages + (long long)page * PAGE * R + ((c / W) * PAGE + t % PAGE) * W + c % W, v);
        }
        store8(out + (long long)row * R + c, v);
    }
}

// x += rms(y) * g; h = x.  One block per row, eight elements per thread and step (at most MAXC steps).  With EXPERTS
// the row y is put together here: sum over the token's experts of weight * output row, plus the gated shared expert.
constexpr int MAXC = 4;
struct Combine {
    const int* at;                 // [N, top] rows of `ye`
    const float* wts;              // [N, top]
    const float* gate;             // [N] or null
    int top;
    long long ye_rows;
};
template <typename T, bool EXPERTS>
__global__ void norm_add_kernel(float* __restrict__ x, const T* __restrict__ y, const T* __restrict__ ys, const float* __restrict__ g,
                                T* __restrict__ h, int D, int width, float eps, Combine cb, int* __restrict__ status) {
    __shared__ float scratch[32];
    kb_dep_trigger();
    kb_dep_wait();
    const long long row = blockIdx.x;
    float v[MAXC][8];
    float ss[1] = {0.f};
    int nc = 0;
    for (int c = threadIdx.x * 8; c < D; c += blockDim.x * 8, ++nc) {
        float* a = v[nc];
        if (!EXPERTS) {
            load8(y + row * D + c, a);
        } else {
#pragma unroll
            for (int j = 0; j < 8; ++j) a[j] = 0.f;
            for (int k = 0; k < cb.top; ++k) {
                const long long r = cb.at[row * cb.top + k];
                const float wk = cb.wts[row * cb.top + k];
                if (r < 0 || r >= cb.ye_rows) {
                    if (c == 0 && status) atomicMax(status, (int)KB_BAD_INDEX);
                    continue;
                }
                float e[8];
                load8(y + r * D + c, e);
#pragma unroll
                for (int j = 0; j < 8; ++j) a[j] += wk * e[j];
            }
            if (ys) {
                const float s = cb.gate ? cb.gate[row] : 1.f;
                float e[8];
                load8(ys + row * D + c, e);
#pragma unroll
                for (int j = 0; j < 8; ++j) a[j] += s * e[j];
            }
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) ss[0] += a[j] * a[j];
    }
    block_sum<1>(ss, scratch);
    const float r = 1.0f / sqrtf(ss[0] / (float)width + eps);
    nc = 0;
    for (int c = threadIdx.x * 8; c < D; c += blockDim.x * 8, ++nc) {
        float xv[8], gv[8];
        load8(x + row * D + c, xv);
        load8(g + c, gv);
#pragma unroll
        for (int j = 0; j < 8; ++j) xv[j] += v[nc][j] * r * gv[j];
        store8(x + row * D + c, xv);
        if ((const void*)h != (const void*)x) store8(h + row * D + c, xv);
    }
}

// x += y (+ step, one vector for all rows); h = rms(x) * w.  One block per row, eight elements per thread and step.  With
// `rows`, output row i is made from row rows[i] and x is left as it is.
template <typename T>
__global__ void __launch_bounds__(1024)
add_norm_kernel(float* __restrict__ x, const T* __restrict__ y, const float* __restrict__ step, const long long* __restrict__ rows,
                const float* __restrict__ w, T* __restrict__ h, int N, int D, int width, float eps, int* __restrict__ status) {
    __shared__ float scratch[32];
    kb_dep_trigger();
    kb_dep_wait();
    long long row = blockIdx.x;
    if (rows) {
        row = rows[row];
        if (row < 0 || row >= N) {                     // uniform over the block
            if (threadIdx.x == 0 && status) atomicMax(status, (int)KB_BAD_INDEX);
            return;
        }
    }
    float v[MAXC][8];
    float ss[1] = {0.f};
#pragma unroll
    for (int i = 0; i < MAXC; ++i) {
        const int c = (i * blockDim.x + threadIdx.x) * 8;
        if (c >= D) break;
        float* a = v[i];
        load8(x + row * D + c, a);
        if (y) {
            float e[8];
            load8(y + row * D + c, e);
#pragma unroll
            for (int j = 0; j < 8; ++j) a[j] += e[j];
        }
        if (step) {
            float e[8];
            load8(step + c, e);
#pragma unroll
            for (int j = 0; j < 8; ++j) a[j] += e[j];
        }
        if (!rows && (y || step)) store8(x + row * D + c, a);
#pragma unroll
        for (int j = 0; j < 8; ++j) ss[0] += a[j] * a[j];
    }
    block_sum<1>(ss, scratch);
    const float r = 1.0f / sqrtf(ss[0] / (float)width + eps);
#pragma unroll
    for (int i = 0; i < MAXC; ++i) {
        const int c = (i * blockDim.x + threadIdx.x) * 8;
        if (c >= D) break;
        float g[8];
        load8(w + c, g);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[i][j] = v[i][j] * r * g[j];
        store8(h + (long long)blockIdx.x * D + c, v[i]);
    }
}

template <typename T>
__global__ void norm_rows_kernel(const float* __restrict__ x, const long long* __restrict__ rows, const float* __restrict__ w,
                                 T* __restrict__ out, int N, int D, int width, float eps, int* __restrict__ status) {
    __shared__ float scratch[32];
    kb_dep_trigger();
    kb_dep_wait();
    const long long src = rows[blockIdx.x], dst = blockIdx.x;
    if (src < 0 || src >= N) {                         // uniform over the block
        if (threadIdx.x == 0 && status) atomicMax(status, (int)KB_BAD_INDEX);
        return;
    }
    float ss[1] = {0.f};
    for (int c = threadIdx.x * 8; c < D; c += blockDim.x * 8) {
        float v[8];
        load8(x + src * D + c, v);
#pragma unroll
        for (int j = 0; j < 8; ++j) ss[0] += v[j] * v[j];
    }
    block_sum<1>(ss, scratch);
    const float r = 1.0f / sqrtf(ss[0] / (float)width + eps);
    for (int c = threadIdx.x * 8; c < D; c += blockDim.x * 8) {
        float v[8], g[8];
        load8(x + src * D + c, v);
        load8(w + c, g);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = v[j] * r * g[j];
        store8(out + dst * D + c, v);
    }
}

// kind 1: exact GELU, kind 2: squared ReLU; n is a multiple of 8
template <typename T>
__global__ void activate_kernel(const T* __restrict__ u, T* __restrict__ out, long long n, int kind) {
    kb_dep_trigger();
    kb_dep_wait();
    for (long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * 8; i < n; i += (long long)gridDim.x * blockDim.x * 8) {
        float v[8];
        load8(u + i, v);
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            if (kind == 1) {
                if constexpr (sizeof(T) == 2) v[j] = gelu_bf16(v[j]);
                else v[j] = 0.5f * v[j] * (1.0f + erff(v[j] * 0.70710678118654752f));
            } else {
                const float p = fmaxf(v[j], 0.f);
                v[j] = p * p;
            }
        }
        store8(out + i, v);
    }
}

// act = silu(gate) * up from rows of gate | up, fp32 (the bf16 form is kb_swiglu_fwd)
__global__ void swiglu_f32_kernel(const float* __restrict__ gu, float* __restrict__ act, long long N, int F) {
    kb_dep_trigger();
    kb_dep_wait();
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < N * F; i += (long long)gridDim.x * blockDim.x) {
        const long long row = i / F, c = i % F;
        const float g = gu[row * 2 * F + c];
        act[i] = g / (1.0f + expf(-g)) * gu[row * 2 * F + F + c];
    }
}

__global__ void softcap_kernel(float* __restrict__ x, long long n, float cap) {
    kb_dep_trigger();
    kb_dep_wait();
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x)
        x[i] = cap * tanhf(x[i] / cap);
}

inline dim3 flat_grid(long long n, int per_block) {
    long long b = (n + per_block - 1) / per_block;
    if (b < 1) b = 1;
    if (b > 148 * 16) b = 148 * 16;
    return dim3((unsigned)b);
}
// threads of a one-block-per-row kernel: one chunk of eight elements each, at most 1024
inline int row_threads(int D) {
    int t = ((D / 8 + 31) / 32) * 32;
    return t > 1024 ? 1024 : (t < 32 ? 32 : t);
}

}  // namespace

// The latent cache is [pages, R / W, 16, W]: W columns of a page's 16 tokens are contiguous.
// Types: 0 = bf16, 1 = fp32 activations.  D and R are multiples of 8, bases 16-byte aligned.
KB_API int kb_embed_pairs(const long long* ids, const int* prev, const void* table, const void* bigram, long long buckets,
                          long long mul_prev, long long mul_cur, float scale, float* x, void* h, int N, int D, int V, int type,
                          int* status, cudaStream_t st) {
    if (D % 8 || N < 1 || V < 1 || (bigram && (buckets < 1 || !prev || mul_prev < 0 || mul_cur < 0))) return 5;
    const dim3 grid = flat_grid((long long)N * (D / 8), 256);
    if (type == 0)
        return kb_launch_dep(embed_pairs_kernel<bf16>, grid, dim3(256), 0, st, ids, prev, (const bf16*)table, (const bf16*)bigram,
                             buckets, mul_prev, mul_cur, scale, x, (bf16*)h, N, D, V, status);
    return kb_launch_dep(embed_pairs_kernel<float>, grid, dim3(256), 0, st, ids, prev, (const float*)table, (const float*)bigram,
                         buckets, mul_prev, mul_cur, scale, x, (float*)h, N, D, V, status);
}
KB_API int kb_latent_append(const void* rows, long long stride, const float* w, int width, float eps, void* pages, int W,
                            const long long* slots, void* out, int N, int R, long long num_slots, int type, int* status,
                            cudaStream_t st) {
    if (R % 8 || stride % 8 || N < 1 || W < 8 || W % 8 || R % W) return 5;
    const dim3 grid((N + 7) / 8);
    if (type == 0)
        return kb_launch_dep(latent_append_kernel<bf16>, grid, dim3(256), 0, st, (const bf16*)rows, stride, w, width, eps,
                             (bf16*)pages, W, slots, (bf16*)out, N, R, num_slots, status);
    return kb_launch_dep(latent_append_kernel<float>, grid, dim3(256), 0, st, (const float*)rows, stride, w, width, eps,
                         (float*)pages, W, slots, (float*)out, N, R, num_slots, status);
}
KB_API int kb_latent_gather(const void* pages, int W, const int* table, int max_pages, const int* cu, int B, void* out, int total, int R,
                            int num_pages, int type, int* status, cudaStream_t st) {
    if (R % 8 || total < 1 || B < 1 || W < 8 || W % 8 || R % W) return 5;
    const dim3 grid = flat_grid((long long)total * (R / 8), 256);
    if (type == 0)
        return kb_launch_dep(latent_gather_kernel<bf16>, grid, dim3(256), 0, st, (const bf16*)pages, W, table, max_pages, cu, B,
                             (bf16*)out, total, R, num_pages, status);
    return kb_launch_dep(latent_gather_kernel<float>, grid, dim3(256), 0, st, (const float*)pages, W, table, max_pages, cu, B,
                         (float*)out, total, R, num_pages, status);
}
// `at` null: y[N, D] is normalised as it is.  Otherwise y holds `ye_rows` expert output rows (see norm_add_kernel).
KB_API int kb_norm_add(float* x, const void* y, const void* ys, const float* g, void* h, int N, int D, int width, float eps,
                       const int* at, const float* wts, const float* gate, int top, long long ye_rows, int type, int* status,
                       cudaStream_t st) {
    if (D % 8 || D > 1024 * 8 * MAXC || N < 1) return 5;
    Combine cb{at, wts, gate, top, ye_rows};
    const dim3 grid(N), block(row_threads(D));
    if (type == 0) {
        if (at)
            return kb_launch_dep(norm_add_kernel<bf16, true>, grid, block, 0, st, x, (const bf16*)y, (const bf16*)ys, g, (bf16*)h, D,
                                 width, eps, cb, status);
        return kb_launch_dep(norm_add_kernel<bf16, false>, grid, block, 0, st, x, (const bf16*)y, (const bf16*)ys, g, (bf16*)h, D,
                             width, eps, cb, status);
    }
    if (at)
        return kb_launch_dep(norm_add_kernel<float, true>, grid, block, 0, st, x, (const float*)y, (const float*)ys, g, (float*)h, D,
                             width, eps, cb, status);
    return kb_launch_dep(norm_add_kernel<float, false>, grid, block, 0, st, x, (const float*)y, (const float*)ys, g, (float*)h, D,
                         width, eps, cb, status);
}
KB_API int kb_norm_rows(const float* x, const long long* rows, const float* w, void* out, int n_rows, int N, int D, int width,
                        float eps, int type, int* status, cudaStream_t st) {
    if (D % 8 || n_rows < 1) return 5;
    if (type == 0)
        return kb_launch_dep(norm_rows_kernel<bf16>, dim3(n_rows), dim3(row_threads(D)), 0, st, x, rows, w, (bf16*)out, N, D, width,
                             eps, status);
    return kb_launch_dep(norm_rows_kernel<float>, dim3(n_rows), dim3(row_threads(D)), 0, st, x, rows, w, (float*)out, N, D, width,
                         eps, status);
}
KB_API int kb_add_norm(float* x, const void* y, const float* step, const long long* rows, const float* w, void* h, int n_rows, int N, int D,
                       int width, float eps, int type, int* status, cudaStream_t st) {
    if (D % 8 || D > 1024 * 8 * MAXC || n_rows < 1) return 5;
    const dim3 grid(n_rows), block(row_threads(D));
    if (type == 0)
        return kb_launch_dep(add_norm_kernel<bf16>, grid, block, 0, st, x, (const bf16*)y, step, rows, w, (bf16*)h, N, D, width, eps,
                             status);
    return kb_launch_dep(add_norm_kernel<float>, grid, block, 0, st, x, (const float*)y, step, rows, w, (float*)h, N, D, width, eps,
                         status);
}
KB_API int kb_swiglu_f32(const float* gu, float* act, long long N, int F, cudaStream_t st) {
    if (N < 1 || F < 1) return 5;
    return kb_launch_dep(swiglu_f32_kernel, flat_grid(N * F, 256), dim3(256), 0, st, gu, act, N, F);
}
KB_API int kb_activate(const void* u, void* out, long long n, int kind, int type, cudaStream_t st) {
    if (n % 8 || (kind != 1 && kind != 2)) return 5;
    const dim3 grid = flat_grid(n / 8, 256);
    if (type == 0) return kb_launch_dep(activate_kernel<bf16>, grid, dim3(256), 0, st, (const bf16*)u, (bf16*)out, n, kind);
    return kb_launch_dep(activate_kernel<float>, grid, dim3(256), 0, st, (const float*)u, (float*)out, n, kind);
}
KB_API int kb_softcap(float* x, long long n, float cap, cudaStream_t st) {
    if (!(cap > 0.f)) return 5;
    return kb_launch_dep(softcap_kernel, flat_grid(n, 256), dim3(256), 0, st, x, n, cap);
}
