// Gated delta rule over whole prompts, 64 tokens at a time on the tensor cores.
//
// Inside a chunk let G_i be the sum of the logarithms of the decays up to token i, L_ij = beta_i e^(G_i - G_j) (k_i . k_j) for
// j < i and A_ij = e^(G_i - G_j) (q_i . k_j) for j <= i.  With the state S in front of the chunk
//
//   T = (I + L)^-1 diag(beta)        R = V - diag(e^G) K S
//   U = T R                          O = diag(e^G) Q S + (A T) R
//   S' = e^(G_64) S + (diag(e^(G_64 - G)) K)^T U
//
// which is the token-by-token recurrence (csrc/delta.cu) solved for the chunk.  Four launches:
//
//   conv      short convolutions + SiLU of q, k and v, to bf16; and the inputs that the next pass's convolutions look back on
//   prepare   one CTA per (chunk, head), all chunks at once: [K; Q] K^T by tcgen05.mma, the unit norms' scalars, L, the inverse (fp32, two
//             32 x 32 triangles by substitution and the block between them), A T by tcgen05.mma; T and A T go to global memory
//   scan      one CTA per (64 value columns, head, sequence) walks the chunks: three tcgen05 products per chunk, [K; Q] S, [T; A T] R
//             and K^T U, each with all 128 rows of the tile in use; the state stays in registers (fp32)
//   finish    output norm and gate
//
// Precision: q, k and v are bf16 after their convolutions and enter the products exactly; their unit norms, like all other
// factors, are fp32 scalars applied to rows of the results.  What is fp32 itself (S, T, A T, R, U) enters as the sum of two bf16
// numbers, so products carry 16 bits of it and sums 24; S is never rounded between chunks.
//
// Every wait is bounded (status word on timeout).  Compiled without fast-math.
#include "attn_common.cuh"
#include "vec.cuh"

namespace {

constexpr int CH = 64;                             // tokens per chunk
constexpr int BLK = CH * 128;                      // a 64-row block of 128-byte rows: 8 KB
constexpr int TT_BYTES = 4 * BLK;                  // [T; A T] upper halves, then lower halves
constexpr int SCALARS = 3 * CH + 8;                // per (chunk, head): e^G r_k | e^G r_q | e^(G_64 - G) r_k | e^G_64
constexpr int LP = 68;                             // pitch (floats) of the fp32 matrices

struct ChunkParams {
    int N, B, H, G, d, dv, dvt, dvp;               // dvt: columns per head of v and o (a multiple of 64), dvp: of the state
    const bf16* rows;                              // projections (beta and decay columns)
    long long stride;
    int col_b, col_a;
    const float *a_log, *dt_bias;
    const int *cu, *ctx, *slots;
    const bf16* v;                                 // [N, H * dvt]
    uint8_t* tt;                                   // [chunk slots, H, TT_BYTES]
    float* scal;                                   // [chunk slots, H, SCALARS]
    float* state;                                  // [num_states, H, d, dvp]
    int num_states;
    bf16* o;                                       // [N, H * dvt]
    int* status;
};

// Chunk c of sequence b has slot cu[b] / 64 + b + c: slots of different sequences never meet, and N / 64 + B of them suffice.
__device__ __forceinline__ int slot_base(const int* cu, int b) { return cu[b] / CH + b; }

__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }

// 64 numbers of a row as two bf16 numbers each, to row `row` of two 128-byte-swizzled tiles
__device__ __forceinline__ void store_row_split(uint8_t* hi, uint8_t* lo, int row, const float* x) {
#pragma unroll
    for (int c = 0; c < 8; ++c) {
        uint32_t h[4], l[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float a = x[c * 8 + 2 * j], b = x[c * 8 + 2 * j + 1];
            const __nv_bfloat162 u = __floats2bfloat162_rn(a, b);
            const float2 f = __bfloat1622float2(u);
            h[j] = *reinterpret_cast<const uint32_t*>(&u);
            l[j] = attn::pack_bf16(a - f.x, b - f.y);
        }
        const int at = row * 128 + ((c ^ (row & 7)) << 4);
        *reinterpret_cast<uint4*>(hi + at) = make_uint4(h[0], h[1], h[2], h[3]);
        *reinterpret_cast<uint4*>(lo + at) = make_uint4(l[0], l[1], l[2], l[3]);
    }
}
__device__ __forceinline__ void tmem_row64(uint32_t taddr, float* x) {
    tc::tmem_ld32(taddr, reinterpret_cast<uint32_t*>(x));
    tc::tmem_ld32(taddr + 32, reinterpret_cast<uint32_t*>(x + 32));
    tc::tmem_ld_wait();
}
__device__ __forceinline__ void bulk_load(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
    asm volatile("cp.async.bulk.shared::cta.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(dst)),
                 "l"(src), "r"(bytes), "r"(smem_u32(bar))
                 : "memory");
}
// The stacked tile [K; Q]: per 64 columns of the head 64 rows of K, then 64 rows of Q.
template <int D>
__device__ __forceinline__ void load_kq(uint8_t* dst, const CUtensorMap* tmK, const CUtensorMap* tmQ, uint64_t* bar, int kvh, int row0) {
    tc::mbar_expect_tx(bar, (D / 64) * 2 * BLK);
#pragma unroll
    for (int h = 0; h < D / 64; ++h) {
        tc::tma_load_3d(dst + h * 2 * BLK, tmK, bar, kvh * D + h * 64, row0, 0);
        tc::tma_load_3d(dst + h * 2 * BLK + BLK, tmQ, bar, kvh * D + h * 64, row0, 0);
    }
}
// d (+)= A B over `STEPS` contraction steps; per step the operands advance by the given bytes (A K-major over 64-column blocks when A_BLK)
template <int STEPS, int A_STEP, int B_STEP, bool A_BLK = false, bool B_BLK = false>
__device__ __forceinline__ void mma_steps(uint32_t d, uint32_t a_addr, uint32_t a_lbo, uint32_t b_addr, uint32_t idesc, bool acc) {
    const tc::DescHalves a = tc::smem_desc_halves(a_addr, a_lbo, 1024), b = tc::smem_desc_halves(b_addr, 16, 1024);
#pragma unroll
    for (int k = 0; k < STEPS; ++k) {
        const uint32_t ao = (A_BLK ? (k >> 2) * 2 * BLK + (k & 3) * A_STEP : k * A_STEP) >> 4;
        const uint32_t bo = (B_BLK ? (k >> 2) * 2 * BLK + (k & 3) * B_STEP : k * B_STEP) >> 4;
        tc::mma_f16_h(d, a.lo + ao, a.hi, b.lo + bo, b.hi, idesc, acc || k > 0);
    }
}

// ------------------------------------------------------------------------------------------------ prepare
constexpr int PREP_SMEM = 4 * BLK + 2 * BLK + CH * LP * 4 + 1024;

template <int D>
__global__ void __launch_bounds__(128)
delta_prepare_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmQ, const ChunkParams p) {
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    uint8_t* sA = smem + 4 * BLK;                      // A, upper and lower half; behind [K; Q], which becomes L and then T
    float* Xs = reinterpret_cast<float*>(sA + 2 * BLK);
    float* Ls = reinterpret_cast<float*>(smem);
    float* M1 = Ls + CH * LP;                          // [32][36]
    uint8_t* sT = smem;
    __shared__ uint64_t bars[2];
    __shared__ uint32_t tmem_slot;
    __shared__ int abort_flag;
    __shared__ float gsum[CH], beta[CH], unit[2 * CH];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int slot = blockIdx.x, head = blockIdx.y, kvh = head / (p.H / p.G);
    int lo = 0, hi = p.B;
    while (hi - lo > 1) {
        const int m = (lo + hi) >> 1;
        if (slot_base(p.cu, m) <= slot) lo = m; else hi = m;
    }
    const int first = p.cu[lo] + (slot - slot_base(p.cu, lo)) * CH;
    const int valid = min(CH, p.cu[lo + 1] - first);
    if (valid <= 0) return;                            // uniform: a slot that no chunk has
    if (tid == 0) {
        tc::mbar_init(&bars[0], 1);
        tc::mbar_init(&bars[1], 1);
        abort_flag = 0;
        tc::fence_barrier_init();
    }
    if (warp == 0) {
        tc::tmem_alloc(&tmem_slot, 128);
        tc::tmem_relinquish();
    }
    tc::tc_fence_before();
    __syncthreads();
    tc::tc_fence_after();
    const uint32_t tmem = tmem_slot;
    bool ok = true;
    if (tid == 0) {
        load_kq<D>(smem, &tmK, &tmQ, &bars[0], kvh, first);
        if (tc::mbar_wait(&bars[0], 0, &abort_flag)) {
            const uint32_t a = smem_u32(smem);
            mma_steps<D / 16, 32, 32, true, true>(tmem, a, 16, a, tc::instr_desc_f16(128, CH, 1, 1, 0, 0), false);
            tc::tc_commit(&bars[1]);
        }
    }
    __syncwarp();
    if (tid < CH) {                                    // decay logarithms (running sum) and step sizes
        float lg = 0.f, be = 0.f;
        if (tid < valid) {
            const bf16* row = p.rows + (long long)(first + tid) * p.stride;
            const float z = to_float(row[p.col_a + head]) + p.dt_bias[head];
            lg = -expf(p.a_log[head]) * (z > 20.f ? z : log1pf(expf(z)));
            be = 1.0f / (1.0f + expf(-to_float(row[p.col_b + head])));
        }
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float t = __shfl_up_sync(0xffffffffu, lg, o);
            if (lane >= o) lg += t;
        }
        gsum[tid] = lg;
        beta[tid] = be;
    }
    ok = tc::mbar_wait(&bars[0], 0, &abort_flag);
    {
        float ss = 0.f;                                // row tid of [K; Q]
#pragma unroll
        for (int h = 0; h < D / 64; ++h)
#pragma unroll
            for (int c = 0; c < 8; ++c) {
                float x[8];
                load8(reinterpret_cast<const bf16*>(smem + h * 2 * BLK + tid * 128 + ((c ^ (tid & 7)) << 4)), x);
#pragma unroll
                for (int j = 0; j < 8; ++j) ss += x[j] * x[j];
            }
        const float r = 1.0f / sqrtf(ss + 1e-6f);
        unit[tid] = (tid & 63) < valid ? (tid < CH ? r : r / sqrtf((float)p.d)) : 0.f;
    }
    ok = tc::mbar_wait(&bars[1], 0, &abort_flag) && ok;
    if (__syncthreads_or(!ok)) {
        if (tid == 0) atomicMax(p.status, (int)KB_TIMEOUT_TMA);
    } else {
        if (tid >= 32 && tid < CH) gsum[tid] += gsum[31];
        __syncthreads();
        tc::tc_fence_after();
        const int i = tid & 63;
        const uint32_t lane_base = (uint32_t)(warp * 32) << 16;
        {
            float x[64];
            tmem_row64(tmem + lane_base, x);
            const float gi = gsum[i], s = tid < CH ? unit[i] * beta[i] : unit[tid];
            const int last = tid < CH ? i - 1 : i;     // columns up to here
#pragma unroll
            for (int j = 0; j < 64; ++j) x[j] = j <= last ? x[j] * s * unit[j] * expf(gi - gsum[j]) : 0.f;
            if (tid < CH) {
#pragma unroll
                for (int j = 0; j < 64; j += 4) *reinterpret_cast<float4*>(Ls + i * LP + j) = make_float4(x[j], x[j + 1], x[j + 2], x[j + 3]);
            } else {
                store_row_split(sA, sA + BLK, i, x);
            }
        }
        __syncthreads();
        // inverses of the two triangles on the diagonal: one column per lane, by substitution
        if (warp < 2) {
            const float* Lb = Ls + (warp * 32) * LP + warp * 32;
            float x[32];
#pragma unroll
            for (int r = 0; r < 32; ++r) {
                float s0 = r == lane ? 1.f : 0.f, s1 = 0.f, s2 = 0.f, s3 = 0.f;
#pragma unroll
                for (int m = 0; m < r; m += 4) {
                    const float4 l4 = *reinterpret_cast<const float4*>(Lb + r * LP + m);
                    s0 = fmaf(-l4.x, x[m], s0);
                    if (m + 1 < r) s1 = fmaf(-l4.y, x[m + 1], s1);
                    if (m + 2 < r) s2 = fmaf(-l4.z, x[m + 2], s2);
                    if (m + 3 < r) s3 = fmaf(-l4.w, x[m + 3], s3);
                }
                x[r] = (s0 + s1) + (s2 + s3);
                Xs[(warp * 32 + r) * LP + warp * 32 + lane] = x[r];
            }
        } else {
            for (int e = tid - 64; e < 32 * 32; e += 64) Xs[(e >> 5) * LP + 32 + (e & 31)] = 0.f;
        }
        __syncthreads();
        // the block below the diagonal: X21 = -X22 (L21 X11); a thread makes eight numbers of a row
        const int r = tid >> 2, c0 = (tid & 3) * 8;
        auto block = [&](const float* Arow, const float* Bm, int pitch, float* acc) {
#pragma unroll
            for (int j = 0; j < 8; ++j) acc[j] = 0.f;
#pragma unroll 8
            for (int m = 0; m < 32; ++m) {
                const float a = Arow[m];
                const float4 b0 = *reinterpret_cast<const float4*>(Bm + m * pitch + c0), b1 = *reinterpret_cast<const float4*>(Bm + m * pitch + c0 + 4);
                acc[0] = fmaf(a, b0.x, acc[0]); acc[1] = fmaf(a, b0.y, acc[1]); acc[2] = fmaf(a, b0.z, acc[2]); acc[3] = fmaf(a, b0.w, acc[3]);
                acc[4] = fmaf(a, b1.x, acc[4]); acc[5] = fmaf(a, b1.y, acc[5]); acc[6] = fmaf(a, b1.z, acc[6]); acc[7] = fmaf(a, b1.w, acc[7]);
            }
        };
        float acc[8];
        block(Ls + (32 + r) * LP, Xs, LP, acc);
#pragma unroll
        for (int j = 0; j < 8; ++j) M1[r * 36 + c0 + j] = acc[j];
        __syncthreads();
        block(Xs + (32 + r) * LP + 32, M1, 36, acc);
#pragma unroll
        for (int j = 0; j < 8; ++j) Xs[(32 + r) * LP + c0 + j] = -acc[j];
        __syncthreads();
        uint8_t* tt = p.tt + ((long long)slot * p.H + head) * TT_BYTES;
        if (tid < CH) {                                // T = X diag(beta)
            float x[64];
#pragma unroll
            for (int j = 0; j < 64; j += 4) {
                const float4 t = *reinterpret_cast<const float4*>(Xs + i * LP + j);
                x[j] = t.x * beta[j];
                x[j + 1] = t.y * beta[j + 1];
                x[j + 2] = t.z * beta[j + 2];
                x[j + 3] = t.w * beta[j + 3];
            }
            store_row_split(sT, sT + BLK, i, x);
        }
        tc::fence_proxy_async();
        tc::tc_fence_before();
        __syncthreads();
        if (tid == 0) {
            tc::tc_fence_after();
            const uint32_t a = smem_u32(sA), t = smem_u32(sT), id = tc::instr_desc_f16(128, CH, 1, 1, 0, 1);
            mma_steps<4, 32, 2048>(tmem + 64, a, 16, t, id, false);            // rows 64 .. 127 of the operand are not looked at
            mma_steps<4, 32, 2048>(tmem + 64, a, 16, t + BLK, id, true);
            mma_steps<4, 32, 2048>(tmem + 64, a + BLK, 16, t, id, true);
            tc::tc_commit(&bars[1]);
        }
        __syncwarp();
        for (int e = tid; e < BLK / 16; e += 128) {
            reinterpret_cast<uint4*>(tt)[e] = reinterpret_cast<const uint4*>(sT)[e];
            reinterpret_cast<uint4*>(tt + 2 * BLK)[e] = reinterpret_cast<const uint4*>(sT + BLK)[e];
        }
        float* sc = p.scal + ((long long)slot * p.H + head) * SCALARS;
        if (tid < CH) {
            const float gi = gsum[tid], gl = gsum[CH - 1];
            sc[tid] = expf(gi) * unit[tid];
            sc[CH + tid] = expf(gi) * unit[CH + tid];
            sc[2 * CH + tid] = expf(gl - gi) * unit[tid];
            if (tid == 0) sc[3 * CH] = gl > -0.5f ? 1.0f + expm1f(gl) : expf(gl);   // as the decays in csrc/delta.cu
        }
        if (tc::mbar_wait(&bars[1], 1, &abort_flag)) {
            tc::tc_fence_after();
            if (warp < 2) {
                float x[64];
                tmem_row64(tmem + 64 + lane_base, x);
                store_row_split(tt + BLK, tt + 3 * BLK, i, x);
            }
        } else if (lane == 0) {
            atomicMax(p.status, (int)KB_TIMEOUT_MMA);
        }
    }
    tc::tc_fence_before();
    __syncthreads();
    if (warp == 0) {
        tc::tc_fence_after();
        tc::tmem_dealloc(tmem, 128);
    }
}

// ------------------------------------------------------------------------------------------------ scan
template <int D>
struct Scan {
    static constexpr int KQ = (D / 64) * 2 * BLK, S_HALF = D * 128;
    static constexpr int OFF_TT = KQ, OFF_S = OFF_TT + TT_BYTES, OFF_RU = OFF_S + 2 * S_HALF, OFF_BAR = OFF_RU + 2 * BLK;
    static constexpr int SMEM = OFF_BAR + 64;
};

template <int D>
__global__ void __launch_bounds__(128, 2)
delta_scan_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmQ, const ChunkParams p) {
    extern __shared__ __align__(1024) uint8_t smem[];
    using L = Scan<D>;
    uint8_t *sKQ = smem, *sTT = smem + L::OFF_TT, *sS = smem + L::OFF_S, *sRU = smem + L::OFF_RU;
    uint64_t* bars = reinterpret_cast<uint64_t*>(smem + L::OFF_BAR);      // [K; Q] loaded, [T; A T] loaded, product done
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 3);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
    const int tid = threadIdx.x, warp = tid >> 5;
    const int tile = blockIdx.x, head = blockIdx.y, b = blockIdx.z, kvh = head / (p.H / p.G);
    const int row0 = p.cu[b], n = p.cu[b + 1] - row0, chunks = (n + CH - 1) / CH;
    if (n <= 0) return;
    if (smem_u32(smem) & 1023) {                       // uniform: the swizzled tiles need this alignment
        if (tid == 0) atomicMax(p.status, (int)KB_BAD_ARG);
        return;
    }
    int slot = p.slots[b];
    if (slot >= p.num_states) {
        if (tid == 0) atomicMax(p.status, (int)KB_BAD_INDEX);
        slot = -1;
    }
    const bool fresh = slot < 0 || p.ctx[b] <= n;
    if (tid == 0) {
        for (int i = 0; i < 3; ++i) tc::mbar_init(bars + i, 1);
        *abort_flag = 0;
        tc::fence_barrier_init();
    }
    if (warp == 0) {
        tc::tmem_alloc(tmem_slot, 256);
        tc::tmem_relinquish();
    }
    tc::tc_fence_before();
    __syncthreads();
    tc::tc_fence_after();
    const uint32_t tmem = *tmem_slot, lane_base = (uint32_t)(warp * 32) << 16;
    const int base = slot_base(p.cu, b);
    const uint8_t* tt = p.tt + ((long long)base * p.H + head) * TT_BYTES;
    const float* sc = p.scal + ((long long)base * p.H + head) * SCALARS;
    if (tid == 0) {
        load_kq<D>(sKQ, &tmK, &tmQ, bars, kvh, row0);
        tc::mbar_expect_tx(bars + 1, TT_BYTES);
        bulk_load(sTT, tt, TT_BYTES, bars + 1);
    }
    __syncwarp();
    // row tid of the state: 64 columns
    float S[64];
    float* st = p.state + (((long long)(slot < 0 ? 0 : slot) * p.H + head) * p.d + tid) * p.dvp + tile * 64;
    const bool own = tid < p.d;
#pragma unroll
    for (int c = 0; c < 64; c += 4) {
        float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
        if (own && !fresh && tile * 64 + c < p.dvp) f = *reinterpret_cast<const float4*>(st + c);
        S[c] = f.x; S[c + 1] = f.y; S[c + 2] = f.z; S[c + 3] = f.w;
    }
    if (tid < D) store_row_split(sS, sS + L::S_HALF, tid, S);
    const int i = tid & 63;
    const uint32_t aKQ = smem_u32(sKQ), aTT = smem_u32(sTT), aS = smem_u32(sS), aRU = smem_u32(sRU);
    const uint32_t id_kb = tc::instr_desc_f16(128, 64, 1, 1, 0, 1), id_mb = tc::instr_desc_f16(128, 64, 1, 1, 1, 1);
    uint32_t done = 0;                                 // parity of the product barrier
    bool failed = false;
    for (int c = 0; c < chunks; ++c) {
        const int at = row0 + c * CH, valid = min(CH, n - c * CH);
        tc::fence_proxy_async();
        tc::tc_fence_before();
        if (__syncthreads_or(failed)) { failed = true; break; }
        if (tid == 0) {                                // X = [K; Q] S
            if (tc::mbar_wait(bars, c & 1, abort_flag)) {
                tc::tc_fence_after();
                mma_steps<D / 16, 32, 2048, true>(tmem, aKQ, 16, aS, id_kb, false);
                mma_steps<D / 16, 32, 2048, true>(tmem, aKQ, 16, aS + L::S_HALF, id_kb, true);
                tc::tc_commit(bars + 2);
            } else {
                failed = true;
            }
        }
        __syncwarp();
        const float* s = sc + (long long)c * p.H * SCALARS;
        const float e = s[tid], eu = s[2 * CH + i], decay = s[3 * CH];
        uint4 v[8];
        if (tid < CH) {
            const uint4* src = reinterpret_cast<const uint4*>(p.v + (long long)(at + i) * p.H * p.dvt + head * p.dvt + tile * 64);
#pragma unroll
            for (int j = 0; j < 8; ++j) v[j] = i < valid ? src[j] : make_uint4(0u, 0u, 0u, 0u);
        }
        failed |= !tc::mbar_wait(bars + 2, done, abort_flag);
        done ^= 1;
        tc::tc_fence_after();
        float x[64];
        tmem_row64(tmem + lane_base, x);
        if (tid < CH) {                                // R = V - e^G r_k X
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                float f[8];
                unpack8(*reinterpret_cast<const bf16x8*>(&v[j]), f);
#pragma unroll
                for (int q = 0; q < 8; ++q) x[j * 8 + q] = fmaf(-e, x[j * 8 + q], f[q]);
            }
            store_row_split(sRU, sRU + BLK, i, x);
        } else {
#pragma unroll
            for (int j = 0; j < 64; ++j) x[j] *= e;
        }
        tc::fence_proxy_async();
        tc::tc_fence_before();
        if (__syncthreads_or(failed)) { failed = true; break; }
        if (tid == 0) {                                // [U; A U] = [T; A T] R
            if (tc::mbar_wait(bars + 1, c & 1, abort_flag)) {
                tc::tc_fence_after();
                mma_steps<4, 32, 2048>(tmem + 64, aTT, 16, aRU, id_kb, false);
                mma_steps<4, 32, 2048>(tmem + 64, aTT, 16, aRU + BLK, id_kb, true);
                mma_steps<4, 32, 2048>(tmem + 64, aTT + 2 * BLK, 16, aRU, id_kb, true);
                tc::tc_commit(bars + 2);
            } else {
                failed = true;
            }
        }
        __syncwarp();
        failed |= !tc::mbar_wait(bars + 2, done, abort_flag);
        done ^= 1;
        tc::tc_fence_after();
        if (tid == 0 && c + 1 < chunks && !failed) {
            tc::mbar_expect_tx(bars + 1, TT_BYTES);
            bulk_load(sTT, tt + (long long)(c + 1) * p.H * TT_BYTES, TT_BYTES, bars + 1);
        }
        __syncwarp();
        {
            float y[64];
            tmem_row64(tmem + 64 + lane_base, y);
            if (tid < CH) {                            // e^(G_64 - G) r_k U
#pragma unroll
                for (int j = 0; j < 64; ++j) y[j] *= eu;
                store_row_split(sRU, sRU + BLK, i, y);
            } else if (i < valid) {
                bf16* dst = p.o + (long long)(at + i) * p.H * p.dvt + head * p.dvt + tile * 64;
#pragma unroll
                for (int j = 0; j < 64; j += 8) {
#pragma unroll
                    for (int q = 0; q < 8; ++q) x[j + q] += y[j + q];
                    store8(dst + j, x + j);
                }
            }
        }
        tc::fence_proxy_async();
        tc::tc_fence_before();
        if (__syncthreads_or(failed)) { failed = true; break; }
        if (tid == 0) {                                // K^T U
            tc::tc_fence_after();
            mma_steps<4, 2048, 2048>(tmem + 128, aKQ, 2 * BLK, aRU, id_mb, false);
            mma_steps<4, 2048, 2048>(tmem + 128, aKQ, 2 * BLK, aRU + BLK, id_mb, true);
            tc::tc_commit(bars + 2);
        }
        __syncwarp();
        failed |= !tc::mbar_wait(bars + 2, done, abort_flag);
        done ^= 1;
        tc::tc_fence_after();
        if (tid == 0 && c + 1 < chunks && !failed) load_kq<D>(sKQ, &tmK, &tmQ, bars, kvh, at + CH);
        __syncwarp();
        tmem_row64(tmem + 128 + lane_base, x);
        if (tid < D) {
#pragma unroll
            for (int j = 0; j < 64; ++j) S[j] = fmaf(decay, S[j], x[j]);
            store_row_split(sS, sS + L::S_HALF, tid, S);
        }
    }
    if (failed) {
        atomicMax(p.status, (int)KB_TIMEOUT_MMA);
        const uint64_t t0 = global_timer_ns();         // copies in flight land before the block's memory is given up
        while (global_timer_ns() - t0 < 2000000ull) {}
    } else if (own && slot >= 0) {
#pragma unroll
        for (int c = 0; c < 64; c += 4)
            if (tile * 64 + c < p.dvp) *reinterpret_cast<float4*>(st + c) = make_float4(S[c], S[c + 1], S[c + 2], S[c + 3]);
    }
    tc::tc_fence_before();
    __syncthreads();
    if (warp == 0) {
        tc::tc_fence_after();
        tc::tmem_dealloc(tmem, 256);
    }
}

// ------------------------------------------------------------------------------------------------ conv, finish
struct ConvParams {
    const bf16* rows;
    long long stride;
    int col_q, col_k, col_v;
    const float* conv;                                 // [2 G d + H dv, taps]
    int N, B, H, G, d, dv, D, dvt;
    bf16* ring;                                        // [num_states, H, ring_rows, 2 d + dv]
    int ring_rows, num_states;
    const int *cu, *ctx, *slots;
    bf16 *q, *k, *v;                                   // [N, G * D], [N, G * D], [N, H * dvt]
};
constexpr int CONV_TOKENS = 32;

// A thread makes eight neighbouring channels of up to CONV_TOKENS neighbouring tokens.
template <int TAPS>
__global__ void __launch_bounds__(128) delta_conv_kernel(const ConvParams p) {
    const int vecs = (2 * p.G * p.d + p.H * p.dv) / 8, vec = blockIdx.y * 128 + threadIdx.x;
    if (vec >= vecs) return;
    const int ch = vec * 8, nq = p.G * p.d;
    int col, ring_head, ring_col, sec = ch < nq ? 0 : ch < 2 * nq ? 1 : 2, in = ch - sec * nq;
    bf16* dst;
    long long dst_stride;
    if (sec < 2) {
        const int g = in / p.d, e = in % p.d;
        col = (sec ? p.col_k : p.col_q) + in;
        ring_head = g * (p.H / p.G);
        ring_col = sec * p.d + e;
        dst = (sec ? p.k : p.q) + g * p.D + e;
        dst_stride = (long long)p.G * p.D;
    } else {
        const int h = in / p.dv, e = in % p.dv;
        col = p.col_v + in;
        ring_head = h;
        ring_col = 2 * p.d + e;
        dst = p.v + h * p.dvt + e;
        dst_stride = (long long)p.H * p.dvt;
    }
    float w[TAPS][8], past[TAPS][8];                   // past[j]: the input j tokens back
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
#pragma unroll
        for (int e = 0; e < 8; ++e) w[j][e] = p.conv[(long long)(ch + e) * TAPS + TAPS - 1 - j];
    const int t0 = blockIdx.x * CONV_TOKENS, t1 = min(p.N, t0 + CONV_TOKENS);
    int b = 0, hi = p.B;
    while (hi - b > 1) {
        const int m = (b + hi) >> 1;
        if (p.cu[m] <= t0) b = m; else hi = m;
    }
    bool enter = true;
    for (int t = t0; t < t1; ++t) {
        while (b + 1 < p.B && t >= p.cu[b + 1]) {
            ++b;
            enter = true;
        }
        if (enter) {
            enter = false;
            const int lo = p.cu[b], n = p.cu[b + 1] - lo, slot = p.slots[b];
            const bool fresh = slot < 0 || slot >= p.num_states || p.ctx[b] <= n;
#pragma unroll
            for (int j = 1; j < TAPS; ++j) {
                if (t - j >= lo) load8(p.rows + (long long)(t - j) * p.stride + col, past[j]);
                else if (!fresh) {
                    // row r of the ring is the input TAPS - 1 - r tokens in front of the pass
                    const bf16* r = p.ring + (((long long)slot * p.H + ring_head) * p.ring_rows + (TAPS - 1 - (j - (t - lo)))) * (2 * p.d + p.dv) + ring_col;
#pragma unroll
                    for (int e = 0; e < 8; ++e) past[j][e] = to_float(r[e]);
                } else {
#pragma unroll
                    for (int e = 0; e < 8; ++e) past[j][e] = 0.f;
                }
            }
        }
        load8(p.rows + (long long)t * p.stride + col, past[0]);
        float z[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) z[e] = past[TAPS - 1][e] * w[TAPS - 1][e];
#pragma unroll
        for (int j = TAPS - 2; j >= 0; --j)
#pragma unroll
            for (int e = 0; e < 8; ++e) z[e] = fmaf(past[j][e], w[j][e], z[e]);
#pragma unroll
        for (int e = 0; e < 8; ++e) z[e] = silu(z[e]);
        store8(dst + (long long)t * dst_stride, z);
#pragma unroll
        for (int j = TAPS - 1; j > 0; --j)
#pragma unroll
            for (int e = 0; e < 8; ++e) past[j][e] = past[j - 1][e];
    }
}

// The convolutions' last inputs, after everything has read the ones before: one block per (head, sequence).
__global__ void __launch_bounds__(256) delta_ring_kernel(const ConvParams p, int taps) {
    extern __shared__ bf16 keep[];                     // [taps - 1, 2 d + dv]
    const int head = blockIdx.x, b = blockIdx.y, kvh = head / (p.H / p.G), C = 2 * p.d + p.dv, past = taps - 1;
    const int lo = p.cu[b], hi = p.cu[b + 1], n = hi - lo, slot = p.slots[b];
    if (n <= 0 || slot < 0 || slot >= p.num_states) return;
    bf16* ring = p.ring + ((long long)slot * p.H + head) * p.ring_rows * C;
    for (int i = threadIdx.x; i < past * C; i += 256) {
        const int c = i % C, at = hi - past + i / C;
        const int col = c < p.d ? p.col_q + kvh * p.d + c : c < 2 * p.d ? p.col_k + kvh * p.d + c - p.d : p.col_v + head * p.dv + c - 2 * p.d;
        keep[i] = at >= lo ? p.rows[(long long)at * p.stride + col] : p.ctx[b] <= n ? __float2bfloat16(0.f) : ring[(past + at - lo) * C + c];
    }
    __syncthreads();
    for (int i = threadIdx.x; i < past * C; i += 256) ring[i] = keep[i];
}

// out = rms(o) * norm * silu(gate): LPH lanes per (token, head)
template <int LPH>
__global__ void __launch_bounds__(256)
delta_finish_kernel(const bf16* __restrict__ o, int dvt, const bf16* __restrict__ gate, long long gate_stride, const float* __restrict__ norm,
                    bf16* __restrict__ out, long long out_stride, long long items, int H, int dv, float eps) {
    const long long item = ((long long)blockIdx.x * 256 + threadIdx.x) / LPH;
    const int sub = threadIdx.x % LPH;
    const bool live = item < items;
    const long long tok = live ? item / H : 0;
    const int head = live ? (int)(item % H) : 0;
    const bf16* src = o + (tok * H + head) * dvt;
    float x[8], ss = 0.f;
    for (int c = sub * 8; live && c < dv; c += LPH * 8) {
        load8(src + c, x);
#pragma unroll
        for (int j = 0; j < 8; ++j) ss += x[j] * x[j];
    }
#pragma unroll
    for (int k = LPH / 2; k > 0; k >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, k);
    const float r = 1.0f / sqrtf(ss / (float)dv + eps);
    for (int c = sub * 8; live && c < dv; c += LPH * 8) {
        float g[8], w[8];
        load8(src + c, x);
        load8(gate + tok * gate_stride + head * dv + c, g);
        load8(norm + c, w);
#pragma unroll
        for (int j = 0; j < 8; ++j) x[j] = x[j] * r * w[j] * silu(g[j]);
        store8(out + tok * out_stride + head * dv + c, x);
    }
}

// [rows, cols] bf16, box 64 columns x 64 rows, 128-byte swizzle
int rows_tmap(CUtensorMap* m, const void* base, long long rows, long long cols) {
    attn::EncodeTiledFn enc = attn::get_encode();
    if (!enc) return 100;
    cuuint64_t dims[3] = {(cuuint64_t)cols, (cuuint64_t)rows, 1};
    cuuint64_t strides[2] = {(cuuint64_t)cols * 2, (cuuint64_t)rows * cols * 2};
    cuuint32_t box[3] = {64, CH, 1}, estr[3] = {1, 1, 1};
    const CUresult r = enc(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                           CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    return r == CUDA_SUCCESS ? 0 : 200 + (int)r;
}
template <typename K>
int allow_smem(K kernel, int bytes, bool* flags) {
    bool* done = kb_device_flag(flags);
    if (!done) return 7;
    if (!*done) {
        if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes) != cudaSuccess) return 7;
        *done = true;
    }
    return 0;
}
template <int D>
int launch_chunks(const ChunkParams& p, const bf16* q, const bf16* k, cudaStream_t st) {
    static bool f1[64] = {}, f2[64] = {};
    int r = allow_smem(delta_prepare_kernel<D>, PREP_SMEM, f1);
    if (!r) r = allow_smem(delta_scan_kernel<D>, Scan<D>::SMEM, f2);
    CUtensorMap tmK, tmQ;
    if (!r) r = rows_tmap(&tmK, k, p.N, (long long)p.G * D);
    if (!r) r = rows_tmap(&tmQ, q, p.N, (long long)p.G * D);
    if (r) return r;
    delta_prepare_kernel<D><<<dim3(p.N / CH + p.B, p.H), 128, PREP_SMEM, st>>>(tmK, tmQ, p);
    delta_scan_kernel<D><<<dim3(p.dvt / 64, p.H, p.B), 128, Scan<D>::SMEM, st>>>(tmK, tmQ, p);
    return kb_launch_status();
}

}  // namespace

// Bytes of `tt` and floats of `scal` for N tokens of B sequences.
KB_API long long kb_delta_chunk_tt_bytes(int N, int B, int H) { return (long long)(N / CH + B) * H * TT_BYTES; }
KB_API long long kb_delta_chunk_scalars(int N, int B, int H) { return (long long)(N / CH + B) * H * SCALARS; }
// Whether the chunked form takes these sizes.
KB_API int kb_delta_chunk_ok(int H, int G, int d, int dv, int taps) {
    return H >= 1 && G >= 1 && H % G == 0 && d >= 8 && d <= 128 && d % 8 == 0 && dv >= 8 && dv % 8 == 0 && taps >= 1 && taps <= 4 &&
           (taps - 1) * (2 * d + dv) * 2 <= 48 * 1024;
}

// rows: projections [N, stride] bf16 (see kb_delta_step); q, k: [N, G, D] with D = 64 or 128 (zeros behind d), v, o: [N, H, dvt] with dvt a
// multiple of 64 (zeros behind dv in v), tt (1024-byte aligned) and scal: workspaces.
KB_API int kb_delta_chunks(const void* rows, long long stride, int col_q, int col_k, int col_v, int col_g, int col_b, int col_a, const float* conv,
                           const float* a_log, const float* dt_bias, const float* norm, int taps, int N, int B, int H, int G, int d, int dv,
                           int D, int dvt, int dvp, float eps, float* state, void* ring, int ring_rows, int num_states, const int* slots,
                           const int* cu, const int* ctx, void* q, void* k, void* v, void* o, void* tt, float* scal, void* out,
                           long long out_stride, int* status, cudaStream_t st) {
    if (!kb_delta_chunk_ok(H, G, d, dv, taps) || N < 1 || B < 1 || B > 65535 || H > 65535 || (D != 64 && D != 128) || d > D || dvt % 64 || dvt < dv ||
        dvp % 4 || dvp < dv || ring_rows < taps - 1 || !slots || !cu || !ctx || !status)
        return 5;
    if (stride % 8 || ((col_q | col_k | col_v | col_g) & 7) || out_stride % 8 || ((uintptr_t)tt & 127)) return 6;
    const ConvParams c{(const bf16*)rows, stride, col_q, col_k, col_v, conv, N, B, H, G, d, dv, D, dvt, (bf16*)ring, ring_rows, num_states,
                       cu, ctx, slots, (bf16*)q, (bf16*)k, (bf16*)v};
    const dim3 grid((N + CONV_TOKENS - 1) / CONV_TOKENS, ((2 * G * d + H * dv) / 8 + 127) / 128);
    if (taps == 1) delta_conv_kernel<1><<<grid, 128, 0, st>>>(c);
    else if (taps == 2) delta_conv_kernel<2><<<grid, 128, 0, st>>>(c);
    else if (taps == 3) delta_conv_kernel<3><<<grid, 128, 0, st>>>(c);
    else delta_conv_kernel<4><<<grid, 128, 0, st>>>(c);
    if (taps > 1) delta_ring_kernel<<<dim3(H, B), 256, (taps - 1) * (2 * d + dv) * 2, st>>>(c, taps);
    if (kb_launch_status()) return KB_LAUNCH_FAILED;
    const ChunkParams p{N, B, H, G, d, dv, dvt, dvp, (const bf16*)rows, stride, col_b, col_a, a_log, dt_bias, cu, ctx, slots, (const bf16*)v,
                        (uint8_t*)tt, scal, state, num_states, (bf16*)o, status};
    const int r = D == 128 ? launch_chunks<128>(p, (const bf16*)q, (const bf16*)k, st) : launch_chunks<64>(p, (const bf16*)q, (const bf16*)k, st);
    if (r) return r;
    const long long items = (long long)N * H;
    const bf16* gate = (const bf16*)rows + col_g;
#define KB_FINISH(LPH) delta_finish_kernel<LPH><<<(unsigned)((items * LPH + 255) / 256), 256, 0, st>>>((const bf16*)o, dvt, gate, stride, norm, \
        (bf16*)out, out_stride, items, H, dv, eps)
    if (dv <= 64) KB_FINISH(8);
    else if (dv <= 128) KB_FINISH(16);
    else KB_FINISH(32);
#undef KB_FINISH
    return kb_launch_status();
}
