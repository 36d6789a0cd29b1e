// Gated delta rule, token by token in fp32: short convolutions + SiLU + unit norms, decay and step size, state update,
// read-out, output norm and gate in one launch, one block per (head, sequence).  Two kernels:
//   step     any number of tokens, the head's state [d, dv] in registers (32-bit mode, short portions)
//   decode   one token: the state is one contiguous piece of memory, copied to shared memory and back by the copy engine, three
//            blocks per SM, so that memory stays busy while other blocks compute
// Compiled without fast-math.
//
//   S = g S;  u = beta (v - S^T k);  S = S + k u^T;  o = S^T q
//
// Both products over the old state are taken in one pass: with a = S^T k, b = S^T q (unscaled S),
//   u = beta (v - g a),   o = g b + (k . q) u,   S = g S + k u^T.
#include "tc.cuh"
#include "vec.cuh"

namespace {

constexpr int THREADS = 256;

struct DeltaParams {
    const void* rows;              // projections of the packed tokens
    long long stride;
    int col_q, col_k, col_v, col_g, col_b, col_a;
    const float* conv;             // [taps, 2 G d + H dv]
    const float *a_log, *dt_bias, *norm;
    int taps, H, G, d, dv, dvp;
    float eps;
    float* state;                  // [num_states, H, d, dvp]
    void* ring;                    // [num_states, H, ring_rows, 2 d + dv], the convolutions' last inputs
    int ring_rows, num_states;
    const int *slots, *cu, *ctx;   // per sequence: state slot, first row (null: row b), tokens so far including these
    void* out;                     // [N, H * dv]
    long long out_stride;
    int* status;
};

__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }
// e^x for x <= 0, rounded to nearest where the result is close to one: a state keeps the product of thousands of these
__device__ __forceinline__ float decay(float x) { return x > -0.5f ? 1.0f + expm1f(x) : expf(x); }
__device__ __forceinline__ float softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// NR: rows of the state per thread (0: the state stays in global memory).  A thread owns four neighbouring columns.
template <typename T, int NR>
__global__ void __launch_bounds__(THREADS, NR > 16 ? 1 : 2)
delta_step_kernel(const DeltaParams p) {
    extern __shared__ float ds_smem[];
    const int C = 2 * p.d + p.dv, past = p.taps - 1;
    float* cur = ds_smem;                              // [C] convolved q | k | v
    float* hist = cur + (C + 3) / 4 * 4;               // [past, C] inputs of the convolutions before the first token
    const int CG = p.dvp / 4;
    int RG = THREADS / CG;
    if (RG > p.d) RG = p.d;
    float* red = hist + (past * C + 3) / 4 * 4;        // [RG, 2, dvp] partial a | b
    float* uo = red + RG * 2 * p.dvp;                  // u [dvp] | o [dvp]
    __shared__ float dots[3];
    kb_dep_trigger();
    const int head = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int kvh = head / (p.H / p.G);
    const int cg = tid % CG, rg = tid / CG;
    const bool owner = rg < RG;
    // The inputs of the pass and this layer run's state were complete before the kernel in front of this one began
    // (nothing else in a pass touches them), so they are fetched before the wait.
    const int lo = p.cu ? p.cu[b] : b, hi = p.cu ? p.cu[b + 1] : b + 1;
    int slot = p.slots[b];
    if (slot >= p.num_states) {
        if (tid == 0 && p.status) atomicMax(p.status, (int)KB_BAD_INDEX);
        slot = -1;
    }
    const bool fresh = slot < 0 || p.ctx[b] <= hi - lo;
    float* st = p.state + ((long long)(slot < 0 ? 0 : slot) * p.H + head) * p.d * p.dvp;
    T* ring = reinterpret_cast<T*>(p.ring) + ((long long)(slot < 0 ? 0 : slot) * p.H + head) * p.ring_rows * C;
    float4 S[NR > 0 ? NR : 1];
    if (NR > 0) {
#pragma unroll
        for (int r = 0; r < NR; ++r) {
            const int i = rg + r * RG;
            S[r] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (owner && i < p.d && !fresh) S[r] = *reinterpret_cast<const float4*>(st + (long long)i * p.dvp + cg * 4);
        }
    }
    for (int i = tid; i < past * C; i += THREADS) hist[i] = fresh ? 0.f : to_float(ring[i]);
    kb_dep_wait();
    const T* rows = reinterpret_cast<const T*>(p.rows);
    const float neg_a = -expf(p.a_log[head]), bias = p.dt_bias[head];
    auto column = [&](int c) { return c < p.d ? p.col_q + kvh * p.d + c : c < 2 * p.d ? p.col_k + kvh * p.d + c - p.d : p.col_v + head * p.dv + c - 2 * p.d; };
    __syncthreads();                                   // hist
    for (int t = lo; t < hi; ++t) {
        const T* row = rows + (long long)t * p.stride;
        const float beta = 1.0f / (1.0f + expf(-to_float(row[p.col_b + head])));
        const float g = decay(neg_a * softplus(to_float(row[p.col_a + head]) + bias));
        for (int c = tid; c < C; c += THREADS) {
            const int col = column(c);
            const int channels = 2 * p.G * p.d + p.H * p.dv;
            const float* w = p.conv + (c < p.d ? kvh * p.d + c : c < 2 * p.d ? (p.G + kvh) * p.d + c - p.d : 2 * p.G * p.d + head * p.dv + c - 2 * p.d);
            float z = 0.f;
            for (int j = 0; j < p.taps; ++j) {
                const int i = t - past + j;            // the tap's token
                z = fmaf(w[(long long)j * channels], i >= lo ? to_float(rows[(long long)i * p.stride + col]) : hist[(past + i - lo) * C + c], z);
            }
            cur[c] = silu(z);
        }
        __syncthreads();
        const float *q = cur, *k = cur + p.d, *v = cur + 2 * p.d;
        if (warp < 3) {                                // q . q, k . k, q . k
            float s = 0.f;
            for (int i = lane; i < p.d; i += 32) s += (warp == 1 ? k[i] : q[i]) * (warp == 0 ? q[i] : k[i]);
            s = warp_sum(s);
            if (lane == 0) dots[warp] = s;
        }
        if (owner) {
            float a[4] = {0.f, 0.f, 0.f, 0.f}, o[4] = {0.f, 0.f, 0.f, 0.f};
            auto add = [&](const float4 s, int i) {
                const float ki = k[i], qi = q[i];
                a[0] = fmaf(s.x, ki, a[0]); a[1] = fmaf(s.y, ki, a[1]); a[2] = fmaf(s.z, ki, a[2]); a[3] = fmaf(s.w, ki, a[3]);
                o[0] = fmaf(s.x, qi, o[0]); o[1] = fmaf(s.y, qi, o[1]); o[2] = fmaf(s.z, qi, o[2]); o[3] = fmaf(s.w, qi, o[3]);
            };
            if (NR > 0) {
#pragma unroll
                for (int r = 0; r < NR; ++r) {
                    const int i = rg + r * RG;
                    if (i < p.d) add(S[r], i);
                }
            } else if (!(fresh && t == lo)) {
                for (int i = rg; i < p.d; i += RG) add(*reinterpret_cast<const float4*>(st + (long long)i * p.dvp + cg * 4), i);
            }
            *reinterpret_cast<float4*>(red + (rg * 2) * p.dvp + cg * 4) = make_float4(a[0], a[1], a[2], a[3]);
            *reinterpret_cast<float4*>(red + (rg * 2 + 1) * p.dvp + cg * 4) = make_float4(o[0], o[1], o[2], o[3]);
        }
        __syncthreads();
        const float rq = 1.0f / sqrtf(dots[0] + 1e-6f) / sqrtf((float)p.d), rk = 1.0f / sqrtf(dots[1] + 1e-6f);
        const float kq = dots[2] * rk * rq;
        for (int c = tid; c < p.dvp; c += THREADS) {
            float a = 0.f, o = 0.f;
            for (int r = 0; r < RG; ++r) {
                a += red[(r * 2) * p.dvp + c];
                o += red[(r * 2 + 1) * p.dvp + c];
            }
            const float u = c < p.dv ? beta * (v[c] - g * rk * a) : 0.f;
            uo[c] = u;
            uo[p.dvp + c] = c < p.dv ? g * rq * o + kq * u : 0.f;
        }
        __syncthreads();
        if (owner) {
            const float4 u = *reinterpret_cast<const float4*>(uo + cg * 4);
            auto step = [&](float4 s, int i) {
                const float ki = k[i] * rk;
                s.x = fmaf(g, s.x, ki * u.x); s.y = fmaf(g, s.y, ki * u.y); s.z = fmaf(g, s.z, ki * u.z); s.w = fmaf(g, s.w, ki * u.w);
                return s;
            };
            if (NR > 0) {
#pragma unroll
                for (int r = 0; r < NR; ++r) {
                    const int i = rg + r * RG;
                    if (i < p.d) {
                        S[r] = step(S[r], i);
                        if (t == hi - 1 && slot >= 0) *reinterpret_cast<float4*>(st + (long long)i * p.dvp + cg * 4) = S[r];
                    }
                }
            } else if (slot >= 0) {
                for (int i = rg; i < p.d; i += RG) {
                    float4* at = reinterpret_cast<float4*>(st + (long long)i * p.dvp + cg * 4);
                    *at = step(fresh && t == lo ? make_float4(0.f, 0.f, 0.f, 0.f) : *at, i);
                }
            }
        }
        float ss = 0.f;                                // every warp sums the whole head: no further barrier
        for (int c = lane; c < p.dv; c += 32) ss += uo[p.dvp + c] * uo[p.dvp + c];
        const float r = 1.0f / sqrtf(warp_sum(ss) / (float)p.dv + p.eps);
        T* dst = reinterpret_cast<T*>(p.out) + (long long)t * p.out_stride + (long long)head * p.dv;
        for (int c = tid; c < p.dv; c += THREADS)
            from_float(dst + c, uo[p.dvp + c] * r * p.norm[c] * silu(to_float(row[p.col_g + head * p.dv + c])));
        __syncthreads();                               // cur, red and uo are written again
    }
    if (slot >= 0)
        for (int i = tid; i < past * C; i += THREADS) {
            const int c = i % C, at = hi - past + i / C;
            from_float(ring + i, at >= lo ? to_float(rows[(long long)at * p.stride + column(c)]) : hist[(past + at - lo) * C + c]);
        }
}

constexpr int MAX_TAPS = 4, MAX_CH = 4;              // decode kernel: taps, channels per thread

template <typename T>
__global__ void __launch_bounds__(THREADS, 3)
delta_decode_kernel(const DeltaParams p) {
    extern __shared__ __align__(16) float dd_smem[];
    const int C = 2 * p.d + p.dv, past = p.taps - 1, CG = p.dvp / 4;
    int RG = THREADS / CG;
    if (RG > p.d) RG = p.d;
    float* Ss = dd_smem;                               // [d, dvp]
    float* cur = Ss + p.d * p.dvp;                     // [C] convolved q | k | v
    float* red = cur + (C + 3) / 4 * 4;                // [RG, 2, dvp]
    float* uo = red + RG * 2 * p.dvp;                  // u [dvp] | o [dvp]
    __shared__ float dots[3];
    __shared__ uint64_t bar;
    __shared__ int abort_flag;
    kb_dep_trigger();
    const int head = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int kvh = head / (p.H / p.G), cg = tid % CG, rg = tid / CG;
    const bool owner = rg < RG;
    // As in the step kernel, what only the passes before this one wrote is fetched before the wait.
    int slot = p.slots[b];
    if (slot >= p.num_states) {
        if (tid == 0 && p.status) atomicMax(p.status, (int)KB_BAD_INDEX);
        slot = -1;
    }
    const bool fresh = slot < 0 || p.ctx[b] <= 1;
    float* st = p.state + ((long long)(slot < 0 ? 0 : slot) * p.H + head) * p.d * p.dvp;
    T* ring = reinterpret_cast<T*>(p.ring) + ((long long)(slot < 0 ? 0 : slot) * p.H + head) * p.ring_rows * C;
    const uint32_t bytes = (uint32_t)(p.d * p.dvp * 4);
    if (tid == 0) {
        tc::mbar_init(&bar, 1);
        abort_flag = 0;
        tc::fence_barrier_init();
        if (!fresh) {
            tc::mbar_expect_tx(&bar, bytes);
            asm volatile("cp.async.bulk.shared::cta.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(Ss)), "l"(st),
                         "r"(bytes), "r"(smem_u32(&bar))
                         : "memory");
        }
    }
    T in[MAX_CH][MAX_TAPS - 1];
    float w[MAX_CH][MAX_TAPS];
    const int channels = 2 * p.G * p.d + p.H * p.dv;
#pragma unroll
    for (int k = 0; k < MAX_CH; ++k) {
        const int c = tid + k * THREADS;
        if (c >= C) break;
        const float* wc = p.conv + (c < p.d ? kvh * p.d + c : c < 2 * p.d ? (p.G + kvh) * p.d + c - p.d : 2 * p.G * p.d + head * p.dv + c - 2 * p.d);
#pragma unroll
        for (int j = 0; j < MAX_TAPS; ++j) w[k][j] = j < p.taps ? wc[(long long)j * channels] : 0.f;
#pragma unroll
        for (int j = 0; j < MAX_TAPS - 1; ++j)
            if (j < past) {
                if (fresh) from_float(&in[k][j], 0.f);
                else in[k][j] = ring[j * C + c];
            }
    }
    const float neg_a = -expf(p.a_log[head]), bias = p.dt_bias[head];
    kb_dep_wait();
    const T* row = reinterpret_cast<const T*>(p.rows) + (long long)b * p.stride;
    const T tb = row[p.col_b + head], ta = row[p.col_a + head];
#pragma unroll
    for (int k = 0; k < MAX_CH; ++k) {
        const int c = tid + k * THREADS;
        if (c >= C) break;
        const T now = row[c < p.d ? p.col_q + kvh * p.d + c : c < 2 * p.d ? p.col_k + kvh * p.d + c - p.d : p.col_v + head * p.dv + c - 2 * p.d];
        float z = 0.f;
#pragma unroll
        for (int j = 0; j < MAX_TAPS; ++j)
            if (j < p.taps) {
                const T x = j < past ? in[k][j < MAX_TAPS - 1 ? j : 0] : now;
                z = fmaf(w[k][j], to_float(x), z);
                if (j > 0 && slot >= 0) ring[(j - 1) * C + c] = x;
            }
        cur[c] = silu(z);
    }
    const float beta = 1.0f / (1.0f + expf(-to_float(tb)));
    const float g = decay(neg_a * softplus(to_float(ta) + bias));
    __syncthreads();
    const float *q = cur, *k = cur + p.d, *v = cur + 2 * p.d;
    if (warp < 3) {                                    // q . q, k . k, q . k
        float s = 0.f;
        for (int i = lane; i < p.d; i += 32) s += (warp == 1 ? k[i] : q[i]) * (warp == 0 ? q[i] : k[i]);
        s = warp_sum(s);
        if (lane == 0) dots[warp] = s;
    }
    const bool ok = fresh || tc::mbar_wait(&bar, 0, &abort_flag);
    if (owner && ok) {
        float a[4] = {0.f, 0.f, 0.f, 0.f}, o[4] = {0.f, 0.f, 0.f, 0.f};
        if (!fresh) {
#pragma unroll 4
            for (int i = rg; i < p.d; i += RG) {
                const float4 s = *reinterpret_cast<const float4*>(Ss + i * p.dvp + cg * 4);
                const float ki = k[i], qi = q[i];
                a[0] = fmaf(s.x, ki, a[0]); a[1] = fmaf(s.y, ki, a[1]); a[2] = fmaf(s.z, ki, a[2]); a[3] = fmaf(s.w, ki, a[3]);
                o[0] = fmaf(s.x, qi, o[0]); o[1] = fmaf(s.y, qi, o[1]); o[2] = fmaf(s.z, qi, o[2]); o[3] = fmaf(s.w, qi, o[3]);
            }
        }
        *reinterpret_cast<float4*>(red + (rg * 2) * p.dvp + cg * 4) = make_float4(a[0], a[1], a[2], a[3]);
        *reinterpret_cast<float4*>(red + (rg * 2 + 1) * p.dvp + cg * 4) = make_float4(o[0], o[1], o[2], o[3]);
    }
    if (__syncthreads_or(!ok)) {                       // the copy did not arrive in time: nothing is written
        if (tid == 0 && p.status) atomicMax(p.status, (int)KB_TIMEOUT_TMA);
        return;
    }
    const float rq = 1.0f / sqrtf(dots[0] + 1e-6f) / sqrtf((float)p.d), rk = 1.0f / sqrtf(dots[1] + 1e-6f);
    const float kq = dots[2] * rk * rq;
    for (int c = tid; c < p.dvp; c += THREADS) {
        float a = 0.f, o = 0.f;
        for (int r = 0; r < RG; ++r) {
            a += red[(r * 2) * p.dvp + c];
            o += red[(r * 2 + 1) * p.dvp + c];
        }
        const float u = c < p.dv ? beta * (v[c] - g * rk * a) : 0.f;
        uo[c] = u;
        uo[p.dvp + c] = c < p.dv ? g * rq * o + kq * u : 0.f;
    }
    __syncthreads();
    if (owner && slot >= 0) {
        const float4 u = *reinterpret_cast<const float4*>(uo + cg * 4);
#pragma unroll 4
        for (int i = rg; i < p.d; i += RG) {
            float4* at = reinterpret_cast<float4*>(Ss + i * p.dvp + cg * 4);
            float4 s = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *at;
            const float ki = k[i] * rk;
            s.x = fmaf(g, s.x, ki * u.x); s.y = fmaf(g, s.y, ki * u.y); s.z = fmaf(g, s.z, ki * u.z); s.w = fmaf(g, s.w, ki * u.w);
            *at = s;
        }
    }
    tc::fence_proxy_async();
    __syncthreads();
    if (tid == 0 && slot >= 0) {
        asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;" ::"l"(st), "r"(smem_u32(Ss)), "r"(bytes) : "memory");
        asm volatile("cp.async.bulk.commit_group;" ::: "memory");
    }
    float ss = 0.f;                                    // every warp sums the whole head: no further barrier
    for (int c = lane; c < p.dv; c += 32) ss += uo[p.dvp + c] * uo[p.dvp + c];
    const float r = 1.0f / sqrtf(warp_sum(ss) / (float)p.dv + p.eps);
    T* dst = reinterpret_cast<T*>(p.out) + (long long)b * p.out_stride + (long long)head * p.dv;
    for (int c = tid; c < p.dv; c += THREADS)
        from_float(dst + c, uo[p.dvp + c] * r * p.norm[c] * silu(to_float(row[p.col_g + head * p.dv + c])));
    if (tid == 0 && slot >= 0) asm volatile("cp.async.bulk.wait_group 0;" ::: "memory");      // the state is read out of shared memory, and written
}

template <typename T, int NR>
int launch_step(const DeltaParams& p, int B, size_t smem, cudaStream_t st) {
    static bool flags[64] = {};
    bool* done = kb_device_flag(flags);
    if (!done) return 7;
    if (!*done) {
        if (cudaFuncSetAttribute(delta_step_kernel<T, NR>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024) != cudaSuccess) return 7;
        *done = true;
    }
    return kb_launch_dep(delta_step_kernel<T, NR>, dim3(p.H, B), dim3(THREADS), smem, st, p);
}
template <typename T>
int dispatch_step(const DeltaParams& p, int B, cudaStream_t st) {
    const int C = 2 * p.d + p.dv, CG = p.dvp / 4;
    int RG = THREADS / CG;
    if (RG > p.d) RG = p.d;
    const int rows = (p.d + RG - 1) / RG;
    const size_t smem = 4 * (size_t)((C + 3) / 4 * 4 + ((p.taps - 1) * C + 3) / 4 * 4 + RG * 2 * p.dvp + 2 * p.dvp);
    if (smem > 160 * 1024) return 5;
    const size_t one = 4 * (size_t)(p.d * p.dvp + (C + 3) / 4 * 4 + RG * 2 * p.dvp + 2 * p.dvp);
    if (!p.cu && p.taps <= MAX_TAPS && C <= MAX_CH * THREADS && one <= 200 * 1024) {
        static bool flags[64] = {};
        bool* done = kb_device_flag(flags);
        if (!done) return 7;
        if (!*done) {
            if (cudaFuncSetAttribute(delta_decode_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess) return 7;
            *done = true;
        }
        return kb_launch_dep(delta_decode_kernel<T>, dim3(p.H, B), dim3(THREADS), one, st, p);
    }
    if (rows <= 4) return launch_step<T, 4>(p, B, smem, st);
    if (rows <= 8) return launch_step<T, 8>(p, B, smem, st);
    if (rows <= 16) return launch_step<T, 16>(p, B, smem, st);
    if (rows <= 32) return launch_step<T, 32>(p, B, smem, st);
    return launch_step<T, 0>(p, B, smem, st);
}

}  // namespace

// rows: projections [N, stride], the parts starting at the given columns; out: [N, out_stride].  Types: 0 = bf16, 1 = fp32 (rows, ring,
// out).  slots[b] < 0: the sequence starts from zero and nothing is kept.
KB_API int kb_delta_step(const void* rows, long long stride, int col_q, int col_k, int col_v, int col_g, int col_b, int col_a, const float* conv,
                         const float* a_log, const float* dt_bias, const float* norm, int taps, int H, int G, int d, int dv, int dvp, float eps,
                         float* state, void* ring, int ring_rows, int num_states, const int* slots, const int* cu, const int* ctx, int B,
                         void* out, long long out_stride, int type, int* status, cudaStream_t st) {
    if (B < 1 || B > 65535 || H < 1 || G < 1 || H % G || d < 1 || dv < 1 || dvp % 4 || dvp < dv || dvp > 4 * THREADS || taps < 1 ||
        ring_rows < taps - 1 || !slots || !ctx)
        return 5;
    const DeltaParams p{rows, stride, col_q, col_k, col_v, col_g, col_b, col_a, conv, a_log, dt_bias, norm, taps, H, G, d, dv, dvp, eps,
                        state, ring, ring_rows, num_states, slots, cu, ctx, out, out_stride, status};
    return type == 0 ? dispatch_step<bf16>(p, B, st) : dispatch_step<float>(p, B, st);
}
