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
//   scan      one CTA per (128 value columns, head, sequence) walks the chunks: three tcgen05 products per chunk; the state stays in
//             registers (fp32)
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
constexpr int LP = 36, TB = 32 * LP;               // pitch and size (floats) of a 32 x 32 fp32 block

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

// 8 * CHUNKS numbers of a row as two bf16 numbers each, from 16-byte chunk `c0` on, to row `row` of two 128-byte-swizzled tiles
template <int CHUNKS>
__device__ __forceinline__ void store_row_split(uint8_t* hi, uint8_t* lo, int row, int c0, const float* x) {
#pragma unroll
    for (int c = 0; c < CHUNKS; ++c) {
        uint32_t h[4], l[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            // the upper half is cut off, the rest (exact) is rounded: integer instructions, where the conversions share the
            // special-function unit
            const uint32_t a = __float_as_uint(x[c * 8 + 2 * j]), b = __float_as_uint(x[c * 8 + 2 * j + 1]);
            h[j] = __byte_perm(a, b, 0x7632);
            const float ra = __uint_as_float(a) - __uint_as_float(a & 0xffff0000u), rb = __uint_as_float(b) - __uint_as_float(b & 0xffff0000u);
            l[j] = __byte_perm(__float_as_uint(ra) + 0x8000u, __float_as_uint(rb) + 0x8000u, 0x7632);
        }
        const int at = row * 128 + (((c0 + c) ^ (row & 7)) << 4);
        *reinterpret_cast<uint4*>(hi + at) = make_uint4(h[0], h[1], h[2], h[3]);
        *reinterpret_cast<uint4*>(lo + at) = make_uint4(l[0], l[1], l[2], l[3]);
    }
}
__device__ __forceinline__ void tmem_row32(uint32_t taddr, float* x) {
    tc::tmem_ld32(taddr, reinterpret_cast<uint32_t*>(x));
    tc::tmem_ld_wait();
}
// 32 columns of the sum of two results 64 columns apart
__device__ __forceinline__ void tmem_sum32(uint32_t taddr, float* x) {
    float y[32];
    tc::tmem_ld32(taddr, reinterpret_cast<uint32_t*>(x));
    tc::tmem_ld32(taddr + 64, reinterpret_cast<uint32_t*>(y));
    tc::tmem_ld_wait();
#pragma unroll
    for (int j = 0; j < 32; ++j) x[j] += y[j];
}
// 2^x by the special-function unit (relative error 2^-22)
__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// z sigmoid(z) where the result is rounded to bf16
__device__ __forceinline__ float silu(float z) {
    float r;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.0f + ex2(-attn::LOG2E * z)));
    return z * r;
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
// d (+)= A B over `STEPS` contraction steps; per step the operands advance by the given bytes (A_BLK, B_BLK: K-major over 64-column
// blocks).  The two halves of an fp32 operand may be one B of 128 columns, `b_lbo` bytes apart; the 64-column results are then added
// when they are read back.
template <int STEPS, int A_STEP, int B_STEP, bool A_BLK = false, bool B_BLK = false>
__device__ __forceinline__ void mma_steps(uint32_t d, uint32_t a_addr, uint32_t a_lbo, uint32_t b_addr, uint32_t b_lbo, uint32_t idesc, bool acc) {
    const tc::DescHalves a = tc::smem_desc_halves(a_addr, a_lbo, 1024), b = tc::smem_desc_halves(b_addr, b_lbo, 1024);
#pragma unroll
    for (int k = 0; k < STEPS; ++k) {
        const uint32_t ao = (A_BLK ? (k >> 2) * 2 * BLK + (k & 3) * A_STEP : k * A_STEP) >> 4;
        const uint32_t bo = (B_BLK ? (k >> 2) * 2 * BLK + (k & 3) * B_STEP : k * B_STEP) >> 4;
        tc::mma_f16_h(d, a.lo + ao, a.hi, b.lo + bo, b.hi, idesc, acc || k > 0);
    }
}

// ------------------------------------------------------------------------------------------------ prepare
// A (16 KB); [K; Q] (32 KB), which gives way to the fp32 blocks of L and X and then to T
constexpr int PREP_SMEM = 6 * BLK + 1024;

// acc = four numbers of a row of a product: sum over m < 16 of A[m] B[m][0 .. 4)
__device__ __forceinline__ void block_row(const float* A, const float* B, float* acc) {
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[j] = 0.f;
#pragma unroll
    for (int m = 0; m < 16; m += 4) {
        const float4 a4 = *reinterpret_cast<const float4*>(A + m);
        const float a[4] = {a4.x, a4.y, a4.z, a4.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const float4 b = *reinterpret_cast<const float4*>(B + (m + e) * LP);
            acc[0] = fmaf(a[e], b.x, acc[0]); acc[1] = fmaf(a[e], b.y, acc[1]); acc[2] = fmaf(a[e], b.z, acc[2]); acc[3] = fmaf(a[e], b.w, acc[3]);
        }
    }
}
// C = s A B for 32 x 32 blocks: thread t < 64 makes a 4 x 4 tile
__device__ __forceinline__ void block_tile(const float* A, const float* B, float* C, float s, int t) {
    const int r0 = (t >> 3) * 4, c0 = (t & 7) * 4;
    float acc[4][4] = {};
#pragma unroll 1
    for (int m = 0; m < 32; m += 4) {
        float a[4][4];
#pragma unroll
        for (int r = 0; r < 4; ++r) *reinterpret_cast<float4*>(a[r]) = *reinterpret_cast<const float4*>(A + (r0 + r) * LP + m);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const float4 b = *reinterpret_cast<const float4*>(B + (m + e) * LP + c0);
#pragma unroll
            for (int r = 0; r < 4; ++r) {
                acc[r][0] = fmaf(a[r][e], b.x, acc[r][0]); acc[r][1] = fmaf(a[r][e], b.y, acc[r][1]);
                acc[r][2] = fmaf(a[r][e], b.z, acc[r][2]); acc[r][3] = fmaf(a[r][e], b.w, acc[r][3]);
            }
        }
    }
#pragma unroll
    for (int r = 0; r < 4; ++r)
        *reinterpret_cast<float4*>(C + (r0 + r) * LP + c0) = make_float4(s * acc[r][0], s * acc[r][1], s * acc[r][2], s * acc[r][3]);
}

template <int D>
__global__ void __launch_bounds__(128, 4)
delta_prepare_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmQ, const ChunkParams p) {
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    uint8_t *sA = smem, *sKQ = smem + 2 * BLK, *sT = sKQ;                  // A and T: upper and lower half
    // blocks (0, 0), (1, 0), (1, 1) of L, a product, and the same blocks of X = (I + L)^-1; T lies over L
    float *Lb = reinterpret_cast<float*>(sKQ), *M1 = Lb + 3 * TB, *Xb = M1 + TB;
    __shared__ uint64_t bars[2];
    __shared__ uint32_t tmem_slot;
    __shared__ int abort_flag;
    __shared__ __align__(16) float gsum[CH], beta[CH], unit[2 * CH]; // sums of log2 of the decays; step sizes; scalars of the unit norms
    const int tid = threadIdx.x, warp = __shfl_sync(0xffffffffu, tid >> 5, 0), lane = tid & 31;    // the warp's number is uniform, and known to be
    const int slot = blockIdx.x, head = blockIdx.y, kvh = head / (p.H / p.G);
    int b = 0;                                         // the last sequence whose slots begin at or in front of this one
    for (int b0 = 0; b0 < p.B; b0 += 32) {
        const unsigned in = __ballot_sync(0xffffffffu, b0 + lane < p.B && slot_base(p.cu, b0 + lane) <= slot);
        if (in) b = b0 + 31 - __clz(in);
        if (in != 0xffffffffu) break;
    }
    const int first = p.cu[b] + (slot - slot_base(p.cu, b)) * CH;
    const int valid = min(CH, p.cu[b + 1] - first);
    if (valid <= 0) return;                            // uniform: a slot that no chunk has
    if (tid == 0) {
        tc::mbar_init(&bars[0], 1);
        tc::mbar_init(&bars[1], 1);
        abort_flag = 0;
        tc::fence_barrier_init();
        load_kq<D>(sKQ, &tmK, &tmQ, &bars[0], kvh, first);
    }
    __syncwarp();
    if (warp == 0) {
        tc::tmem_alloc(&tmem_slot, 128);
        tc::tmem_relinquish();
    }
    if (tid >= 64) {                                   // decays (running sum) and step sizes of the tokens
        const int t = tid - 64;
        float lg = 0.f, be = 0.f;
        if (t < valid) {
            const bf16* row = p.rows + (long long)(first + t) * p.stride;
            const float z = to_float(row[p.col_a + head]) + p.dt_bias[head];
            lg = -expf(p.a_log[head]) * (z > 20.f ? z : log1pf(expf(z))) * attn::LOG2E;
            be = 1.0f / (1.0f + expf(-to_float(row[p.col_b + head])));
        }
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float u = __shfl_up_sync(0xffffffffu, lg, o);
            if (lane >= o) lg += u;
        }
        gsum[t] = lg;
        beta[t] = be;
    }
    tc::tc_fence_before();
    __syncthreads();
    tc::tc_fence_after();
    const uint32_t tmem = __shfl_sync(0xffffffffu, tmem_slot, 0), lane_base = (uint32_t)(warp * 32) << 16;
    bool ok = tc::mbar_wait(&bars[0], 0, &abort_flag);
    // Products are issued by one elected lane of a whole warp: their operands then stay in uniform registers.
    if (warp == 0 && __all_sync(0xffffffffu, ok)) {
        const uint32_t a = smem_u32(sKQ);
        if (tc::elect_one()) {
            mma_steps<D / 16, 32, 32, true, true>(tmem, a, 16, a, 16, tc::instr_desc_f16(128, CH, 1, 1, 0, 0), false);
            tc::tc_commit(&bars[1]);
        }
        __syncwarp();
    }
    {
        float ss = 0.f;                                // row tid of [K; Q]
#pragma unroll
        for (int h = 0; h < D / 64; ++h)
#pragma unroll
            for (int c = 0; c < 8; ++c) {
                float x[8];
                load8(reinterpret_cast<const bf16*>(sKQ + h * 2 * BLK + tid * 128 + ((c ^ (tid & 7)) << 4)), x);
#pragma unroll
                for (int j = 0; j < 8; ++j) ss += x[j] * x[j];
            }
        const float r = 1.0f / sqrtf(ss + 1e-6f);
        unit[tid] = (tid & 63) < valid ? (tid < CH ? r : r / sqrtf((float)p.d)) : 0.f;
    }
    ok = tc::mbar_wait(&bars[1], 0, &abort_flag) && ok;
    if (tid >= 32 && tid < CH) gsum[tid] += gsum[31];
    if (__syncthreads_or(!ok)) {
        if (tid == 0) atomicMax(p.status, (int)KB_TIMEOUT_TMA);
    } else {
        tc::tc_fence_after();
        const int i = tid & 63;
        // (loops are kept rolled where they can be: four blocks per SM at different places share the instruction cache)
#pragma unroll 1
        for (int h = 0; h < 64; h += 32) {
            float x[32];
            tmem_row32(tmem + lane_base + h, x);
            const float gi = gsum[i], s = tid < CH ? unit[i] * beta[i] : unit[tid];
            const int last = (tid < CH ? i - 1 : i) - h;                   // columns up to here
#pragma unroll
            for (int j = 0; j < 32; j += 4) {
                const float4 u = *reinterpret_cast<const float4*>(unit + h + j), g = *reinterpret_cast<const float4*>(gsum + h + j);
                x[j] = j <= last ? x[j] * s * u.x * ex2(gi - g.x) : 0.f;
                x[j + 1] = j + 1 <= last ? x[j + 1] * s * u.y * ex2(gi - g.y) : 0.f;
                x[j + 2] = j + 2 <= last ? x[j + 2] * s * u.z * ex2(gi - g.z) : 0.f;
                x[j + 3] = j + 3 <= last ? x[j + 3] * s * u.w * ex2(gi - g.w) : 0.f;
            }
            if (tid < CH) {
                if (h == 0 || i >= 32) {
                    float* dst = Lb + (i < 32 ? 0 : h ? 2 * TB : TB) + (i & 31) * LP;
#pragma unroll
                    for (int j = 0; j < 32; j += 4) *reinterpret_cast<float4*>(dst + j) = make_float4(x[j], x[j + 1], x[j + 2], x[j + 3]);
                }
            } else {
                store_row_split<4>(sA, sA + BLK, i, h >> 3, x);
            }
            __syncwarp();
        }
        __syncthreads();
        // inverses of the four 16 x 16 triangles on the diagonal, one per warp: a column per lane, by substitution
        {
            const int off = (warp >> 1) * 2 * TB + (warp & 1) * (16 * LP + 16);
            const float* Lw = Lb + off;
            float* Xw = Xb + off;
            float x[16];
#pragma unroll
            for (int r = 0; r < 16; ++r) {
                float s0 = r == lane ? 1.f : 0.f, s1 = 0.f, s2 = 0.f, s3 = 0.f;
#pragma unroll
                for (int m = 0; m < r; m += 4) {
                    const float4 l4 = *reinterpret_cast<const float4*>(Lw + r * LP + m);
                    s0 = fmaf(-l4.x, x[m], s0);
                    if (m + 1 < r) s1 = fmaf(-l4.y, x[m + 1], s1);
                    if (m + 2 < r) s2 = fmaf(-l4.z, x[m + 2], s2);
                    if (m + 3 < r) s3 = fmaf(-l4.w, x[m + 3], s3);
                }
                x[r] = (s0 + s1) + (s2 + s3);
                // lanes 16 .. 31 hold zeros: above the diagonal in an even block's rows, nothing in an odd block's
                if (lane < 16 || !(warp & 1)) Xw[r * LP + lane] = x[r];
            }
        }
        __syncthreads();
        {                                              // below the diagonal of each 32 x 32 block: X21 = -X22 (L21 X11), 16 x 16
            const int off = (tid >> 6) * 2 * TB, r = (tid & 63) >> 2, c0 = (tid & 3) * 4;
            float acc[4];
            block_row(Lb + off + (16 + r) * LP, Xb + off + c0, acc);
            float* m = M1 + (tid >> 6) * 16 * LP;
            *reinterpret_cast<float4*>(m + r * LP + c0) = make_float4(acc[0], acc[1], acc[2], acc[3]);
            __syncthreads();
            block_row(Xb + off + (16 + r) * LP + 16, m + c0, acc);
            *reinterpret_cast<float4*>(Xb + off + (16 + r) * LP + c0) = make_float4(-acc[0], -acc[1], -acc[2], -acc[3]);
        }
        __syncthreads();
        // and of the whole, 32 x 32: a 4 x 4 tile per thread of two warps
        if (tid < 64) block_tile(Lb + TB, Xb, M1, 1.f, tid);
        __syncthreads();
        if (tid < 64) block_tile(Xb + 2 * TB, M1, Xb + TB, -1.f, tid);
        __syncthreads();
        uint8_t* tt = p.tt + ((long long)slot * p.H + head) * TT_BYTES;
        {                                              // T = X diag(beta): half a row per thread
            const int r = tid >> 1, hf = tid & 1;
            float x[32];
            const float* src = Xb + (r < 32 ? 0 : (1 + hf) * TB) + (r & 31) * LP;
#pragma unroll
            for (int j = 0; j < 32; j += 4) {
                float4 t = *reinterpret_cast<const float4*>(src + j);
                const float4 be = *reinterpret_cast<const float4*>(beta + hf * 32 + j);
                if (r < 32 && hf) t = make_float4(0.f, 0.f, 0.f, 0.f);
                x[j] = t.x * be.x;
                x[j + 1] = t.y * be.y;
                x[j + 2] = t.z * be.z;
                x[j + 3] = t.w * be.w;
            }
            store_row_split<4>(sT, sT + BLK, r, hf * 4, x);
        }
        tc::fence_proxy_async();
        tc::tc_fence_before();
        __syncthreads();
        if (warp == 0) {
            tc::tc_fence_after();
            const uint32_t a = smem_u32(sA), t = smem_u32(sT);
            // the operand's rows 64 .. 127 (what follows in shared memory) give rows that are not looked at
            if (tc::elect_one()) {
                mma_steps<4, 32, 2048>(tmem, a, 16, t, BLK, tc::instr_desc_f16(128, 128, 1, 1, 0, 1), false);
                mma_steps<4, 32, 2048>(tmem, a + BLK, 16, t, 16, tc::instr_desc_f16(128, 64, 1, 1, 0, 1), true);
                tc::tc_commit(&bars[1]);
            }
            __syncwarp();
        }
        for (int e = tid; e < BLK / 16; e += 128) {
            reinterpret_cast<uint4*>(tt)[e] = reinterpret_cast<const uint4*>(sT)[e];
            reinterpret_cast<uint4*>(tt + 2 * BLK)[e] = reinterpret_cast<const uint4*>(sT + BLK)[e];
        }
        float* sc = p.scal + ((long long)slot * p.H + head) * SCALARS;
        if (tid < CH) {
            const float gi = gsum[tid], gl = gsum[CH - 1];
            sc[tid] = ex2(gi) * unit[tid];
            sc[CH + tid] = ex2(gi) * unit[CH + tid];
            sc[2 * CH + tid] = ex2(gl - gi) * unit[tid];
            if (tid == 0) {                            // the state's own factor: to nearest, as the decays in csrc/delta.cu
                const float x = gl * attn::LN2;
                sc[3 * CH] = x > -0.5f ? 1.0f + expm1f(x) : expf(x);
            }
        }
        if (tc::mbar_wait(&bars[1], 1, &abort_flag)) {
            tc::tc_fence_after();
            if (warp < 2) {
#pragma unroll 1
                for (int h = 0; h < 2; ++h) {
                    float x[32];
                    tmem_sum32(tmem + lane_base + h * 32, x);
                    store_row_split<4>(tt + BLK, tt + 3 * BLK, i, h * 4, x);
                }
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
// The products are taken transposed, with the value columns as the 128 rows of the tile: what a product needs of the state, of R and
// of U is then in the very lanes of tensor memory where the product before left it, and goes back there as its A operand (two bf16
// halves); shared memory holds only what the copy engine brings ([K; Q], [T; A T], V and the scalars of two chunks).
//
//   MMA1  X^T = S^T [K; Q]^T     128 x 128 (tokens of K | tokens of Q)
//   MMA2  [U; A U]^T = R^T [T; A T]^T
//   MMA3  U^T K                  128 x D, added to the decayed state
//
// Sixteen warps, each a quarter of the lanes and of the columns: 16 tokens in K's part of X and U (where R and U are made), the same
// 16 tokens in Q's part (where O is made), 32 rows of the state.  Warp 0 also issues the products, warp 15 the copies.  O leaves
// through shared memory.
template <int D>
struct Scan {
    static constexpr int KQ = (D / 64) * 2 * BLK, OFF_TT = KQ, OFF_V = OFF_TT + TT_BYTES, OFF_SC = OFF_V + 2 * BLK;
    static constexpr int STAGE = OFF_SC + 1024, OFF_O = 2 * STAGE, OFF_BAR = OFF_O + 2 * BLK, SMEM = OFF_BAR + 1024 + 128;
};
constexpr int SCAN_WARPS = 16;

// 2 P numbers as two bf16 numbers each into P + P columns of packed pairs (an A operand in tensor memory)
template <int P>
__device__ __forceinline__ void tmem_store_split(uint32_t hi, uint32_t lo, const float* x) {
    uint32_t h[P], l[P];
#pragma unroll
    for (int j = 0; j < P; ++j) {
        const uint32_t a = __float_as_uint(x[2 * j]), b = __float_as_uint(x[2 * j + 1]);
        h[j] = __byte_perm(a, b, 0x7632);
        const float ra = __uint_as_float(a) - __uint_as_float(a & 0xffff0000u), rb = __uint_as_float(b) - __uint_as_float(b & 0xffff0000u);
        l[j] = __byte_perm(__float_as_uint(ra) + 0x8000u, __float_as_uint(rb) + 0x8000u, 0x7632);
    }
    if constexpr (P == 16) {
        tc::tmem_st16(hi, h);
        tc::tmem_st16(lo, l);
    } else {
        tc::tmem_st8(hi, h);
        tc::tmem_st8(lo, l);
    }
}
__device__ __forceinline__ void scale16(float* x, const float* f) {
#pragma unroll
    for (int j = 0; j < 16; j += 4) {
        const float4 a = *reinterpret_cast<const float4*>(f + j);
        x[j] *= a.x; x[j + 1] *= a.y; x[j + 2] *= a.z; x[j + 3] *= a.w;
    }
}
// d (+)= A B with A in tensor memory (8 columns per step of 16) and B stepped by the given bytes (B_BLK: K-major over 64-column blocks)
template <int STEPS, int B_STEP, bool B_BLK = false>
__device__ __forceinline__ void mma_ts_steps(uint32_t d, uint32_t a_tmem, uint32_t b_addr, uint32_t b_lbo, uint32_t idesc, bool acc) {
    const tc::DescHalves b = tc::smem_desc_halves(b_addr, b_lbo, 1024);
#pragma unroll
    for (int k = 0; k < STEPS; ++k) {
        const uint32_t bo = (B_BLK ? (k >> 2) * 2 * BLK + (k & 3) * B_STEP : k * B_STEP) >> 4;
        tc::mma_f16_ts_h(d, a_tmem + 8 * k, b.lo + bo, b.hi, idesc, acc || k > 0);
    }
}

template <int D>
__global__ void __launch_bounds__(SCAN_WARPS * 32, 1)
delta_scan_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmV,
                  const __grid_constant__ CUtensorMap tmO, const ChunkParams p) {
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    using L = Scan<D>;
    uint64_t* full = reinterpret_cast<uint64_t*>(smem + L::OFF_BAR);      // [2] a chunk's data is there
    uint64_t *ready = full + 2, *done = full + 3;      // the next product's operand is there; a product is done
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(full + 4);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
    const int tid = threadIdx.x, warp = __shfl_sync(0xffffffffu, tid >> 5, 0);
    const int tile = blockIdx.x, head = blockIdx.y, b = blockIdx.z, kvh = head / (p.H / p.G);
    const int row0 = p.cu[b], n = p.cu[b + 1] - row0, chunks = (n + CH - 1) / CH;
    if (n <= 0) return;
    const int base = slot_base(p.cu, b);
    const uint8_t* tt = p.tt + ((long long)base * p.H + head) * TT_BYTES;
    const float* sc = p.scal + ((long long)base * p.H + head) * SCALARS;
    const int boxes = tile * 128 + 64 < p.dvt ? 2 : 1;
    auto load = [&](int c) {                           // one thread
        uint8_t* st = smem + (c & 1) * L::STAGE;
        uint64_t* bar = full + (c & 1);
        const int at = row0 + c * CH;
        tc::mbar_expect_tx(bar, (D / 64) * 2 * BLK + TT_BYTES + boxes * BLK + SCALARS * 4);
#pragma unroll
        for (int h = 0; h < D / 64; ++h) {
            tc::tma_load_3d(st + h * 2 * BLK, &tmK, bar, kvh * D + h * 64, at, 0);
            tc::tma_load_3d(st + h * 2 * BLK + BLK, &tmQ, bar, kvh * D + h * 64, at, 0);
        }
        bulk_load(st + L::OFF_TT, tt + (long long)c * p.H * TT_BYTES, TT_BYTES, bar);
        for (int h = 0; h < boxes; ++h) tc::tma_load_3d(st + L::OFF_V + h * BLK, &tmV, bar, head * p.dvt + tile * 128 + h * 64, at, 0);
        bulk_load(st + L::OFF_SC, sc + (long long)c * p.H * SCALARS, SCALARS * 4, bar);
    };
    if (warp == 0) {
        if (tc::elect_one()) {
            tc::mbar_init(full, 1);
            tc::mbar_init(full + 1, 1);
            tc::mbar_init(ready, SCAN_WARPS);
            tc::mbar_init(done, 1);
            *abort_flag = 0;
            tc::fence_barrier_init();
            load(0);
            if (chunks > 1) load(1);
        }
        __syncwarp();
        tc::tmem_alloc(tmem_slot, 256);
        tc::tmem_relinquish();
    }
    int slot = p.slots[b];
    if (slot >= p.num_states) {
        if (tid == 0) atomicMax(p.status, (int)KB_BAD_INDEX);
        slot = -1;
    }
    const bool fresh = slot < 0 || p.ctx[b] <= n;
    tc::tc_fence_before();
    __syncthreads();
    tc::tc_fence_after();
    // columns 0 .. 127 results; 128 .. 255 the state's two halves as an operand, which R's and U's lie over
    const uint32_t tmem = __shfl_sync(0xffffffffu, *tmem_slot, 0);
    const uint32_t op_hi = tmem + 128, s_lo = op_hi + D / 2, ru_lo = op_hi + 32;
    bool ok = true;
    const int lane = tid & 31, dvi = (warp & 3) * 32 + lane, g = warp >> 2, col = tile * 128 + dvi;
    const bool owns = g * 32 < D;
    const uint32_t lanes = (uint32_t)((warp & 3) * 32) << 16;
    const uint32_t res_k = tmem + lanes + g * 16, res_q = res_k + CH, res_s = tmem + lanes + g * 32;
    const uint32_t s_hi_w = op_hi + lanes + g * 16, s_lo_w = s_lo + lanes + g * 16, ru_hi_w = op_hi + lanes + g * 8, ru_lo_w = ru_lo + lanes + g * 8;
    const uint32_t id1 = tc::instr_desc_f16(128, 128, 1, 1, 0, 0), id3 = tc::instr_desc_f16(128, D, 1, 1, 0, 1);
    uint8_t* sO = smem + L::OFF_O;                     // [2][64 tokens][64 columns]
    uint16_t* o_out = reinterpret_cast<uint16_t*>(sO + (dvi >> 6) * BLK) + g * 16 * 64 + (dvi & 63);
    // S^T: this thread holds value column `col`, rows g * 32 .. of the state
    float S[32];
    float* st = p.state + ((long long)(slot < 0 ? 0 : slot) * p.H + head) * p.d * p.dvp + col;
#pragma unroll
    for (int j = 0; j < 32; ++j) {
        const int i = g * 32 + j;
        S[j] = !fresh && i < p.d && col < p.dvp ? st[(long long)i * p.dvp] : 0.f;
    }
    uint32_t par_ready = 0, par_done = 0;
    auto hand_over = [&]() {                           // what this warp wrote to tensor memory may be multiplied
        tc::tmem_st_wait();
        tc::tc_fence_before();
        __syncwarp();
        if (lane == 0) tc::mbar_arrive(ready);
    };
    auto operand = [&]() {                             // warp 0: every warp has handed over
        ok = tc::mbar_wait(ready, par_ready, abort_flag) && ok;
        par_ready ^= 1;
        tc::tc_fence_after();
    };
    auto issuer = [&]() -> bool {                      // one lane issues; the operands stay in uniform registers
        return __all_sync(0xffffffffu, ok) && tc::elect_one();
    };
    auto result = [&]() {
        __syncwarp();
        ok = tc::mbar_wait(done, par_done, abort_flag) && ok;
        par_done ^= 1;
        tc::tc_fence_after();
    };
    auto store_o = [&](int c) {                        // one thread: the chunk's rows of O (all 64 of them) leave shared memory
        for (int h = 0; h < boxes; ++h)
            asm volatile("cp.async.bulk.tensor.3d.global.shared::cta.tile.bulk_group [%0, {%2, %3, %4}], [%1];" ::"l"(reinterpret_cast<uint64_t>(&tmO)),
                         "r"(smem_u32(sO + h * BLK)), "r"(head * p.dvt + tile * 128 + h * 64), "r"(row0 + c * CH), "r"(0)
                         : "memory");
        asm volatile("cp.async.bulk.commit_group;" ::: "memory");
    };
    if (owns) tmem_store_split<16>(s_hi_w, s_lo_w, S);
    hand_over();
    for (int c = 0; c < chunks; ++c) {
        const uint8_t* sm = smem + (c & 1) * L::STAGE;
        const uint32_t aKQ = smem_u32(smem) + (c & 1) * L::STAGE, aTT = aKQ + L::OFF_TT;
        const float* scal = reinterpret_cast<const float*>(sm + L::OFF_SC);
        ok = tc::mbar_wait(full + (c & 1), (c >> 1) & 1, abort_flag) && ok;
        float x[16], y[16];
        uint32_t v[8];                                 // V, transposed on the way: one number per token, two of them per register
        {
            const uint16_t* src = reinterpret_cast<const uint16_t*>(sm + L::OFF_V + (dvi >> 6) * BLK) + g * 16 * 64 + (dvi & 63);
#pragma unroll
            for (int j = 0; j < 8; ++j) v[j] = (uint32_t)src[2 * j * 64] | (uint32_t)src[(2 * j + 1) * 64] << 16;
        }
        if (warp == 0) {                               // X^T
            operand();
            if (issuer()) {
                mma_ts_steps<D / 16, 32, true>(tmem, op_hi, aKQ, 16, id1, false);
                mma_ts_steps<D / 16, 32, true>(tmem, s_lo, aKQ, 16, id1, true);
                tc::tc_commit(done);
            }
            __syncwarp();
            if (lane == 0 && c > 0 && ok) store_o(c - 1);
        }
        result();
        tc::tmem_ld16(res_k, reinterpret_cast<uint32_t*>(x));
        tc::tmem_ld16(res_q, reinterpret_cast<uint32_t*>(y));
        tc::tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 16; j += 4) {              // R = V - e^G r_k X
            const float4 f = *reinterpret_cast<const float4*>(scal + g * 16 + j);
            x[j] = fmaf(-f.x, x[j], __uint_as_float(v[j / 2] << 16));
            x[j + 1] = fmaf(-f.y, x[j + 1], __uint_as_float(v[j / 2] & 0xffff0000u));
            x[j + 2] = fmaf(-f.z, x[j + 2], __uint_as_float(v[j / 2 + 1] << 16));
            x[j + 3] = fmaf(-f.w, x[j + 3], __uint_as_float(v[j / 2 + 1] & 0xffff0000u));
        }
        tmem_store_split<8>(ru_hi_w, ru_lo_w, x);
        hand_over();
        if (warp == 0) {                               // [U; A U]^T
            operand();
            if (lane == 0) asm volatile("cp.async.bulk.wait_group.read 0;" ::: "memory");     // O's buffer is free when this product is done
            __syncwarp();
            if (issuer()) {
                mma_ts_steps<4, 32>(tmem, op_hi, aTT, 16, id1, false);
                mma_ts_steps<4, 32>(tmem, ru_lo, aTT, 16, id1, true);
                mma_ts_steps<4, 32>(tmem, op_hi, aTT + 2 * BLK, 16, id1, true);
                tc::tc_commit(done);
            }
        } else if (warp == SCAN_WARPS - 1) {           // the chunk before this one is done with its stage
            if (lane == 0 && c > 0 && c + 1 < chunks && ok) load(c + 1);
        }
        scale16(y, scal + CH + g * 16);                // e^G r_q X
        result();
        tc::tmem_ld16(res_k, reinterpret_cast<uint32_t*>(x));
        float z[16];
        tc::tmem_ld16(res_q, reinterpret_cast<uint32_t*>(z));
        tc::tmem_ld_wait();
        scale16(x, scal + 2 * CH + g * 16);            // e^(G_64 - G) r_k U
        tmem_store_split<8>(ru_hi_w, ru_lo_w, x);
        hand_over();
        if (warp == 0) {                               // U^T K
            operand();
            if (issuer()) {
                mma_ts_steps<4, 2048>(tmem, op_hi, aKQ, 2 * BLK, id3, false);
                mma_ts_steps<4, 2048>(tmem, ru_lo, aKQ, 2 * BLK, id3, true);
                tc::tc_commit(done);
            }
            __syncwarp();
        }
        // O = e^G r_q X + A U, while the product runs
        const int valid = n - c * CH;
        if (valid >= CH) {
#pragma unroll
            for (int j = 0; j < 16; ++j) o_out[j * 64] = __bfloat16_as_ushort(__float2bfloat16(y[j] + z[j]));
            tc::fence_proxy_async();
        } else if (col < p.dvt) {                      // the rows behind the sequence's end are another's
            bf16* dst = p.o + (long long)(row0 + c * CH) * p.H * p.dvt + head * p.dvt + col;
#pragma unroll
            for (int j = 0; j < 16; ++j)
                if (g * 16 + j < valid) dst[(long long)(g * 16 + j) * p.H * p.dvt] = __float2bfloat16(y[j] + z[j]);
        }
        const float decay = scal[3 * CH];
        result();
        if (owns) {
            tc::tmem_ld16(res_s, reinterpret_cast<uint32_t*>(x));
            tc::tmem_ld16(res_s + 16, reinterpret_cast<uint32_t*>(y));
            tc::tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 16; ++j) {
                S[j] = fmaf(decay, S[j], x[j]);
                S[16 + j] = fmaf(decay, S[16 + j], y[j]);
            }
            tmem_store_split<16>(s_hi_w, s_lo_w, S);
        }
        hand_over();
        if (!__all_sync(0xffffffffu, ok)) break;
    }
    if (warp == 0 && __all_sync(0xffffffffu, ok)) {    // the last arrivals, before the block ends
        operand();
        if (lane == 0 && ok) {
            if (n % CH == 0) store_o(chunks - 1);
            asm volatile("cp.async.bulk.wait_group 0;" ::: "memory");
        }
        __syncwarp();
    }
    if (ok && slot >= 0 && col < p.dvp) {
#pragma unroll
        for (int j = 0; j < 32; ++j)
            if (g * 32 + j < p.d) st[(long long)(g * 32 + j) * p.dvp] = S[j];
    }
    if (!ok) {
        atomicMax(p.status, (int)KB_TIMEOUT_MMA);
        const uint64_t t0 = global_timer_ns();         // copies in flight land before the block's memory is given up
        while (global_timer_ns() - t0 < 2000000ull) {}
    }
    __syncwarp();
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
    const float* conv;                                 // [taps, 2 G d + H dv]
    int N, B, H, G, d, dv, D, dvt;
    bf16* ring;                                        // [num_states, H, ring_rows, 2 d + dv]
    int ring_rows, num_states;
    const int *cu, *ctx, *slots;
    bf16 *q, *k, *v;                                   // [N, G * D], [N, G * D], [N, H * dvt]
};
constexpr int CONV_TOKENS = 32, CONV_GROUP = 8;

// A thread makes eight neighbouring channels of up to CONV_TOKENS neighbouring tokens; the inputs of CONV_GROUP tokens are fetched together.
template <int TAPS>
__global__ void __launch_bounds__(128, 4) delta_conv_kernel(const ConvParams p) {
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
    for (int j = 0; j < TAPS; ++j) load8(p.conv + (long long)(TAPS - 1 - j) * (2 * nq + p.H * p.dv) + ch, w[j]);
    const int t0 = blockIdx.x * CONV_TOKENS, t1 = min(p.N, t0 + CONV_TOKENS);
    int b = 0, hi = p.B;
    while (hi - b > 1) {
        const int m = (b + hi) >> 1;
        if (p.cu[m] <= t0) b = m; else hi = m;
    }
    int next = b + 1 < p.B ? p.cu[b + 1] : p.N;
    // the inputs in front of token t, which is the first of this thread's or of its sequence
    auto enter = [&](int t) {
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
    };
    auto token = [&](int t, const uint4& in) {
        unpack8(*reinterpret_cast<const bf16x8*>(&in), past[0]);
        float z[8];
#pragma unroll
        for (int e = 0; e < 8; e += 2) {
            float2 a = __fmul2_rn(make_float2(past[TAPS - 1][e], past[TAPS - 1][e + 1]), make_float2(w[TAPS - 1][e], w[TAPS - 1][e + 1]));
#pragma unroll
            for (int j = TAPS - 2; j >= 0; --j) a = __ffma2_rn(make_float2(past[j][e], past[j][e + 1]), make_float2(w[j][e], w[j][e + 1]), a);
            z[e] = silu(a.x);
            z[e + 1] = silu(a.y);
        }
        store8(dst + (long long)t * dst_stride, z);
#pragma unroll
        for (int j = TAPS - 1; j > 0; --j)
#pragma unroll
            for (int e = 0; e < 8; ++e) past[j][e] = past[j - 1][e];
    };
    enter(t0);
    for (int tg = t0; tg < t1; tg += CONV_GROUP) {
        uint4 in8[CONV_GROUP];
#pragma unroll
        for (int u = 0; u < CONV_GROUP; ++u)
            if (tg + u < t1) in8[u] = *reinterpret_cast<const uint4*>(p.rows + (long long)(tg + u) * p.stride + col);
        if (tg + CONV_GROUP <= min(next, t1)) {        // inside one sequence
#pragma unroll
            for (int u = 0; u < CONV_GROUP; ++u) token(tg + u, in8[u]);
        } else {
#pragma unroll
            for (int u = 0; u < CONV_GROUP; ++u) {
                if (tg + u >= t1) break;
                if (tg + u >= next) {
                    while (b + 1 < p.B && tg + u >= next) {
                        ++b;
                        next = b + 1 < p.B ? p.cu[b + 1] : p.N;
                    }
                    enter(tg + u);
                }
                token(tg + u, in8[u]);
            }
        }
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
    const bf16* gsrc = gate + tok * gate_stride + head * dv;
    bf16* dst = out + tok * out_stride + head * dv;
    const int c0 = sub * 8;
    const bool in = live && c0 < dv;
    float x[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f}, g[8], w[8], ss = 0.f;
    if (in) {
        load8(src + c0, x);
        load8(gsrc + c0, g);
        load8(norm + c0, w);
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += x[j] * x[j];
    for (int c = c0 + LPH * 8; live && c < dv; c += LPH * 8) {
        float y[8];
        load8(src + c, y);
#pragma unroll
        for (int j = 0; j < 8; ++j) ss += y[j] * y[j];
    }
#pragma unroll
    for (int k = LPH / 2; k > 0; k >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, k);
    const float r = 1.0f / sqrtf(ss / (float)dv + eps);
    if (!in) return;
#pragma unroll
    for (int j = 0; j < 8; ++j) x[j] = x[j] * r * w[j] * silu(g[j]);
    store8(dst + c0, x);
    for (int c = c0 + LPH * 8; c < dv; c += LPH * 8) {
        load8(src + c, x);
        load8(gsrc + c, g);
        load8(norm + c, w);
#pragma unroll
        for (int j = 0; j < 8; ++j) x[j] = x[j] * r * w[j] * silu(g[j]);
        store8(dst + c, x);
    }
}

// [rows, cols] bf16, box 64 columns x 64 rows
int rows_tmap(CUtensorMap* m, const void* base, long long rows, long long cols, CUtensorMapSwizzle swizzle) {
    attn::EncodeTiledFn enc = attn::get_encode();
    if (!enc) return 100;
    cuuint64_t dims[3] = {(cuuint64_t)cols, (cuuint64_t)rows, 1};
    cuuint64_t strides[2] = {(cuuint64_t)cols * 2, (cuuint64_t)rows * cols * 2};
    cuuint32_t box[3] = {64, CH, 1}, estr[3] = {1, 1, 1};
    const CUresult r = enc(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                           swizzle, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
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
    CUtensorMap tmK, tmQ, tmV, tmO;
    if (!r) r = rows_tmap(&tmK, k, p.N, (long long)p.G * D, CU_TENSOR_MAP_SWIZZLE_128B);
    if (!r) r = rows_tmap(&tmQ, q, p.N, (long long)p.G * D, CU_TENSOR_MAP_SWIZZLE_128B);
    if (!r) r = rows_tmap(&tmV, p.v, p.N, (long long)p.H * p.dvt, CU_TENSOR_MAP_SWIZZLE_NONE);
    if (!r) r = rows_tmap(&tmO, p.o, p.N, (long long)p.H * p.dvt, CU_TENSOR_MAP_SWIZZLE_NONE);
    if (r) return r;
    delta_prepare_kernel<D><<<dim3(p.N / CH + p.B, p.H), 128, PREP_SMEM, st>>>(tmK, tmQ, p);
    delta_scan_kernel<D><<<dim3((p.dvt + 127) / 128, p.H, p.B), SCAN_WARPS * 32, Scan<D>::SMEM, st>>>(tmK, tmQ, tmV, tmO, p);
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
