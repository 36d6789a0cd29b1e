// Grouped attention over paged keys and values whose head sizes are free: rotary positions + unit RMS of the query and
// key heads with the cache append, a packed copy of cached rows, and the attention itself in its plain form (one block per
// token and head, an online softmax over tiles of 128 keys) for the 32-bit mode and for sizes the tensor-core kernels do
// not take.  Compiled without fast-math.
#include "vec.cuh"

namespace {

constexpr int PAGE = 16, TILE = 128, MAXE = 8;         // value sizes up to TILE * MAXE

struct HeadShape {
    int H, G, dim, vdim;                               // heads and sizes in the projection's rows
    int kd, vd;                                        // sizes in the cache and in the packed rows (zeros behind dim, vdim)
    int half;                                          // rotated pairs: (i, i + half)
    int col_k, col_v;                                  // first columns of the key and value parts
};

// A walk item is one (token, head); heads are H query heads, then G key heads, then G value heads (copied only).
// VEC: LPH lanes share a head; a lane owns one pair of eight-element chunks (both halves of the rotation) or one chunk behind
// the rotated part.  Otherwise a warp takes a head, element by element.
template <typename T, bool VEC, int LPH>
__global__ void __launch_bounds__(256)
head_rotary_kernel(const T* __restrict__ rows, long long stride, const HeadShape s, const float* __restrict__ cosT,
                   const float* __restrict__ sinT, int positions_max, const int* __restrict__ positions, float eps, T* __restrict__ q,
                   T* __restrict__ k, T* __restrict__ v, T* __restrict__ k_pages, T* __restrict__ v_pages,
                   const long long* __restrict__ slots, long long num_slots, int N, int* __restrict__ status) {
    kb_dep_trigger();
    kb_dep_wait();
    constexpr int HPW = 32 / LPH;
    const int lane = threadIdx.x & 31, sub = lane % LPH;
    const int heads = s.H + 2 * s.G;
    const long long items = (long long)N * heads;
    const long long nwarps = (long long)gridDim.x * (blockDim.x >> 5);
    for (long long base = ((long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5)) * HPW; base < items; base += nwarps * HPW) {
        const long long item = base + lane / LPH;
        const bool live = item < items;
        const long long tok = live ? item / heads : 0;
        const int hd = live ? (int)(item % heads) : 0;
        const bool isq = hd < s.H, isv = hd >= s.H + s.G;
        const int kvh = isv ? hd - s.H - s.G : hd - s.H;
        const T* src = rows + tok * stride + (isq ? hd * s.dim : isv ? s.col_v + kvh * s.vdim : s.col_k + kvh * s.dim);
        int pos = positions[tok];
        if (pos < 0 || pos >= positions_max) {
            if (live && sub == 0 && status) atomicMax(status, (int)KB_BAD_INDEX);
            pos = 0;
        }
        long long slot = isq ? -1 : slots[tok];
        if (slot >= num_slots) {
            if (live && sub == 0 && status) atomicMax(status, (int)KB_BAD_INDEX);
            slot = -1;
        }
        const int size = isv ? s.vdim : s.dim, padded = isv ? s.vd : s.kd;
        T* dst = isq ? q + (tok * s.H + hd) * s.kd : isv ? (v ? v + (tok * s.G + kvh) * s.vd : nullptr)
                                                         : (k ? k + (tok * s.G + kvh) * s.kd : nullptr);
        T* page = nullptr;
        if (slot >= 0) {
            const long long at = ((slot / PAGE) * s.G + kvh) * PAGE + slot % PAGE;
            page = isv ? v_pages + at * s.vd : k_pages + at * s.kd;
        }
        if constexpr (VEC) {
            const int pairs = s.half / 8, tasks = isv ? s.vdim / 8 : pairs + (s.dim / 8 - 2 * pairs);
            const bool mine = live && sub < tasks, two = !isv && sub < pairs;
            const int c0 = isv ? sub * 8 : two ? sub * 8 : (sub + pairs) * 8;
            float a[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f}, b[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
            if (mine) {
                load8(src + c0, a);
                if (two) {
                    float c[8], sn[8];
                    load8(src + s.half + c0, b);
                    load8(cosT + (long long)pos * s.half + c0, c);
                    load8(sinT + (long long)pos * s.half + c0, sn);
#pragma unroll
                    for (int j = 0; j < 8; ++j) {
                        const float u = a[j], w = b[j];
                        a[j] = u * c[j] - w * sn[j];
                        b[j] = w * c[j] + u * sn[j];
                    }
                }
            }
            float ss = 0.f;
#pragma unroll
            for (int j = 0; j < 8; ++j) ss += a[j] * a[j] + b[j] * b[j];
#pragma unroll
            for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            const float r = isv ? 1.f : 1.0f / sqrtf(ss / (float)s.dim + eps);
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                a[j] *= r;
                b[j] *= r;
            }
            if (mine) {
                if (dst) {
                    store8(dst + c0, a);
                    if (two) store8(dst + s.half + c0, b);
                }
                if (page) {
                    store8(page + c0, a);
                    if (two) store8(page + s.half + c0, b);
                }
            }
            if (live && dst) {
                const float z[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
                for (int c = size + sub * 8; c < padded; c += LPH * 8) store8(dst + c, z);
            }
        } else {
            const float* ct = cosT + (long long)pos * s.half;
            const float* st = sinT + (long long)pos * s.half;
            auto value = [&](int i) -> float {
                const float x = to_float(src[i]);
                if (isv || i >= 2 * s.half) return x;
                if (i < s.half) return x * ct[i] - to_float(src[i + s.half]) * st[i];
                return x * ct[i - s.half] + to_float(src[i - s.half]) * st[i - s.half];
            };
            float ss = 0.f;
            if (live)
                for (int i = lane; i < size; i += 32) {
                    const float x = value(i);
                    ss += x * x;
                }
            ss = warp_sum(ss);
            const float r = isv ? 1.f : 1.0f / sqrtf(ss / (float)s.dim + eps);
            if (live)
                for (int i = lane; i < padded; i += 32) {
                    const float x = i < size ? value(i) * r : 0.f;
                    if (dst) from_float(dst + i, x);
                    if (page) from_float(page + i, x);
                }
        }
    }
}

// Rows of cached positions, packed: segment g holds positions first[g] .. of sequence seq[g] in rows cu[g] .. cu[g + 1].
template <typename T>
__global__ void kv_gather_kernel(const T* __restrict__ k_pages, const T* __restrict__ v_pages, int G, int kd, int vd,
                                 const int* __restrict__ table, int B, int max_pages, int num_pages, const int* __restrict__ seq,
                                 const int* __restrict__ first, const int* __restrict__ cu, int segs, T* __restrict__ k, T* __restrict__ v,
                                 int total, int* __restrict__ status) {
    kb_dep_trigger();
    kb_dep_wait();
    const int kc = kd >> 3, vc = vd >> 3, per = G * (kc + vc);
    const long long n = (long long)total * per;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
        const int row = (int)(i / per), c = (int)(i % per);
        int lo = 0, hi = segs;                         // the segment with cu[lo] <= row < cu[lo + 1]
        while (hi - lo > 1) {
            const int m = (lo + hi) >> 1;
            if (cu[m] <= row) lo = m; else hi = m;
        }
        const int p = first[lo] + row - cu[lo], b = seq[lo], pi = p / PAGE;
        const int page = b >= 0 && b < B && pi >= 0 && pi < max_pages ? table[(long long)b * max_pages + pi] : -1;
        const bool isv = c >= G * kc;
        const int e = isv ? c - G * kc : c, w = isv ? vc : kc, g = e / w, col = (e % w) * 8, size = isv ? vd : kd;
        float x[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
        if (page < 0 || page >= num_pages) {
            if (c == 0 && status) atomicMax(status, (int)KB_BAD_INDEX);
        } else {
            load8((isv ? v_pages : k_pages) + (((long long)page * G + g) * PAGE + p % PAGE) * size + col, x);
        }
        store8((isv ? v : k) + ((long long)row * G + g) * size + col, x);
    }
}

template <typename T>
__global__ void __launch_bounds__(TILE)
paged_attn_kernel(const T* __restrict__ q, const T* __restrict__ k_pages, const T* __restrict__ v_pages, int G, int kd, int vd,
                  const int* __restrict__ table, int max_pages, int num_pages, const int* __restrict__ ctx_lens, const int* __restrict__ cu,
                  int B, const T* __restrict__ gate, long long gate_stride, T* __restrict__ out, int H, int vdim, int cols, float scale,
                  float softcap, int chunk, int* __restrict__ status) {
    extern __shared__ float pa_smem[];
    float* qs = pa_smem;                               // [kd]
    float* ps = qs + kd;                               // [TILE]
    int* at = reinterpret_cast<int*>(ps + TILE);       // [TILE] cache row of every key of the tile, -1: none
    __shared__ float red[2][TILE / 32];
    kb_dep_trigger();
    kb_dep_wait();
    const int n = blockIdx.x, head = blockIdx.y, t = threadIdx.x, lane = t & 31, warp = t >> 5;
    const int kvh = head / (H / G);
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
    const int begin = chunk > 0 ? (keys - 1) / chunk * chunk : 0;
    const T* qrow = q + ((long long)n * H + head) * kd;
    for (int i = t; i < kd; i += TILE) qs[i] = to_float(qrow[i]);
    float o[MAXE];
#pragma unroll
    for (int i = 0; i < MAXE; ++i) o[i] = 0.f;
    float m = -INFINITY, l = 0.f;
    for (int k0 = begin; k0 < keys; k0 += TILE) {
        const int key = k0 + t;
        int row = -1;
        if (key < keys) {
            const int page = table[(long long)b * max_pages + key / PAGE];
            if (page >= 0 && page < num_pages) row = (page * G + kvh) * PAGE + key % PAGE;
            else if (status) atomicMax(status, (int)KB_BAD_INDEX);
        }
        __syncthreads();                               // qs is there; the previous tile's ps and at are done with
        at[t] = row;
        float s = -INFINITY;
        if (row >= 0) {
            const T* kr = k_pages + (long long)row * kd;
            s = 0.f;
            for (int i = 0; i < kd; i += 8) {
                float c[8];
                load8(kr + i, c);
#pragma unroll
                for (int j = 0; j < 8; ++j) s = fmaf(qs[i + j], c[j], s);
            }
            s *= scale;
            if (softcap > 0.f) s = softcap * tanhf(s / softcap);
        }
        const float wm = warp_max(s);
        if (lane == 0) red[0][warp] = wm;
        __syncthreads();
        float mn = m;
#pragma unroll
        for (int w = 0; w < TILE / 32; ++w) mn = fmaxf(mn, red[0][w]);
        const float p = row >= 0 ? expf(s - mn) : 0.f;
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
            if (r >= vdim) break;
            float a = o[i] * f;
            for (int j = 0; j < nk; ++j)
                if (at[j] >= 0) a = fmaf(ps[j], to_float(v_pages[(long long)at[j] * vd + r]), a);
            o[i] = a;
        }
    }
    float g = 1.f;
    if (gate) g = 1.0f / (1.0f + expf(-to_float(gate[(long long)n * gate_stride + head])));
    T* dst = out + ((long long)n * H + head) * cols;
#pragma unroll
    for (int i = 0; i < MAXE; ++i) {
        const int r = i * TILE + t;
        if (r < cols) from_float(dst + r, r < vdim && l > 0.f ? o[i] / l * g : 0.f);
    }
}

template <typename T>
int launch_rotary(const void* rows, long long stride, const HeadShape& s, const float* cosT, const float* sinT, int pmax,
                  const int* positions, float eps, void* q, void* k, void* v, void* kp, void* vp, const long long* slots, long long num_slots,
                  int N, int* status, cudaStream_t st) {
    const long long items = (long long)N * (s.H + 2 * s.G);
    const int pairs = s.half / 8, tasks = s.vdim / 8 > s.dim / 8 - pairs ? s.vdim / 8 : s.dim / 8 - pairs;
    const bool vec = s.half % 8 == 0 && s.dim % 8 == 0 && s.vdim % 8 == 0 && s.kd % 8 == 0 && s.vd % 8 == 0 && stride % 8 == 0 && tasks <= 32 &&
                     s.col_k % 8 == 0 && s.col_v % 8 == 0;
    const int lph = !vec ? 32 : tasks <= 8 ? 8 : tasks <= 16 ? 16 : 32;
    long long blocks = (items * lph + 255) / 256;
    if (blocks > 148 * 32) blocks = 148 * 32;
#define KB_ROT(VEC, LPH) kb_launch_dep(head_rotary_kernel<T, VEC, LPH>, dim3((unsigned)blocks), dim3(256), 0, st, (const T*)rows, stride, s, cosT, \
        sinT, pmax, positions, eps, (T*)q, (T*)k, (T*)v, (T*)kp, (T*)vp, slots, num_slots, N, status)
    if (!vec) return KB_ROT(false, 32);
    return lph == 8 ? KB_ROT(true, 8) : lph == 16 ? KB_ROT(true, 16) : KB_ROT(true, 32);
#undef KB_ROT
}

}  // namespace

// Pages are [num_pages, G, 16, kd] and [num_pages, G, 16, vd].  Types: 0 = bf16, 1 = fp32.  k, v may be null (not kept packed).
KB_API int kb_head_rotary(const void* rows, long long stride, int H, int G, int dim, int vdim, int kd, int vd, int half, int col_k, int col_v,
                          const float* cosT, const float* sinT, int positions_max, const int* positions, float eps, void* q, void* k, void* v,
                          void* k_pages, void* v_pages, const long long* slots, long long num_slots, int N, int type, int* status,
                          cudaStream_t st) {
    if (N < 1 || H < 1 || G < 1 || dim < 1 || vdim < 1 || kd < dim || vd < vdim || half < 0 || 2 * half > dim) return 5;
    const HeadShape s{H, G, dim, vdim, kd, vd, half, col_k, col_v};
    if (type == 0)
        return launch_rotary<bf16>(rows, stride, s, cosT, sinT, positions_max, positions, eps, q, k, v, k_pages, v_pages, slots, num_slots, N,
                                   status, st);
    return launch_rotary<float>(rows, stride, s, cosT, sinT, positions_max, positions, eps, q, k, v, k_pages, v_pages, slots, num_slots, N,
                                status, st);
}
KB_API int kb_kv_gather(const void* k_pages, const void* v_pages, int G, int kd, int vd, const int* table, int B, int max_pages, int num_pages,
                        const int* seq, const int* first, const int* cu, int segs, void* k, void* v, int total, int type, int* status,
                        cudaStream_t st) {
    if (G < 1 || kd % 8 || vd % 8 || segs < 1 || total < 1 || B < 1) return 5;
    long long blocks = ((long long)total * G * ((kd + vd) / 8) + 255) / 256;
    if (blocks > 148 * 32) blocks = 148 * 32;
    if (type == 0)
        return kb_launch_dep(kv_gather_kernel<bf16>, dim3((unsigned)blocks), dim3(256), 0, st, (const bf16*)k_pages, (const bf16*)v_pages, G, kd,
                             vd, table, B, max_pages, num_pages, seq, first, cu, segs, (bf16*)k, (bf16*)v, total, status);
    return kb_launch_dep(kv_gather_kernel<float>, dim3((unsigned)blocks), dim3(256), 0, st, (const float*)k_pages, (const float*)v_pages, G, kd,
                         vd, table, B, max_pages, num_pages, seq, first, cu, segs, (float*)k, (float*)v, total, status);
}
// q: [N, H, kd]; out: [N, H, cols], cols >= vdim; cu null: row n is sequence n.  softcap <= 0: none; chunk <= 0: all keys up to the
// query; gate null: none, else gate[n * gate_stride + head].
KB_API int kb_paged_attn_plain(const void* q, const void* k_pages, const void* v_pages, int G, int kd, int vd, const int* table, int max_pages,
                               int num_pages, const int* ctx_lens, const int* cu, int B, const void* gate, long long gate_stride, void* out,
                               int N, int H, int vdim, int cols, float scale, float softcap, int chunk, int type, int* status,
                               cudaStream_t st) {
    if (N < 1 || H < 1 || H > 65535 || G < 1 || H % G || B < 1 || kd % 8 || kd > 8192 || vdim > vd || cols < vdim || cols > TILE * MAXE ||
        (long long)num_pages * G * PAGE > 0x7fffffffll)
        return 5;
    const size_t smem = (size_t)(kd + 2 * TILE) * 4;
    if (type == 0)
        return kb_launch_dep(paged_attn_kernel<bf16>, dim3(N, H), dim3(TILE), smem, st, (const bf16*)q, (const bf16*)k_pages,
                             (const bf16*)v_pages, G, kd, vd, table, max_pages, num_pages, ctx_lens, cu, B, (const bf16*)gate, gate_stride,
                             (bf16*)out, H, vdim, cols, scale, softcap, chunk, status);
    return kb_launch_dep(paged_attn_kernel<float>, dim3(N, H), dim3(TILE), smem, st, (const float*)q, (const float*)k_pages,
                         (const float*)v_pages, G, kd, vd, table, max_pages, num_pages, ctx_lens, cu, B, (const float*)gate, gate_stride,
                         (float*)out, H, vdim, cols, scale, softcap, chunk, status);
}
