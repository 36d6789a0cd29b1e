// Attention over paged latents for sm_100a: decoding, and short portions of prompts.
// A sequence caches one latent row c[t] of R numbers per token, which every head uses as key and as value, so a pass
// needs each cached row once for all heads.  With the roles of a usual attention turned around - cached tokens on the M
// side of the tensor-core tile, (token, head) query columns on the N side - no tile row is wasted on heads that are
// not there:
//
//   S^T[128 tokens x HG]   = C[128 x R] . Q^T             A = the latent tile K-major,  B = queries  (both in shared memory)
//   O^T[R x HG]           += C^T[R x 128] . P[128 x HG]   A = the same tile MN-major,   B = probabilities
//
// The cache keeps a page as blocks of 64 latent columns, [R / 64][16 tokens][64]: a block is 2 KB of contiguous memory.
// The tile is fetched by TMA block by block (128-byte swizzle) into a ring of slots of 128
// tokens x 128 latent columns; it stays there from the first product to the second.  S^T and O^T live in tensor memory.  A
// thread of the softmax warps owns one token of the tile; a column's maximum is a warp reduction plus an exchange
// through shared memory, refreshed lazily (O^T is rescaled only when a maximum grows by more than 2^8).
//
// Work: a unit is (sequence, group of HG query columns), its tiles are the 128-token tiles of the context that the
// group sees; one CTA per SM.  With no more units than SMs every unit is cut into pieces of at most P tiles, P being the
// smallest number for which there are no more pieces than SMs, and a CTA takes one piece (piece g writes partial g).
// Otherwise all units' tiles form one line that is cut into equal parts, one per CTA; the part that CTA g has of unit u
// writes partial g + u.  The pieces of a unit are put together by a merge kernel.
// Roles (256 threads): warps 0 and 6 = TMA of the latents (one half of a slot each: a lane issues one page, and issuing
// is what a single warp would be bound by), warp 7 = TMA of the queries, warp 1 = MMA issue and TMEM owner, warps 2-5 = softmax and output.
// While the softmax of a tile runs, the tensor pipe already works on the scores of the next one, as far as the ring
// holds it.
// All waits are bounded (status word on timeout).
#include <cuda.h>

#include "tc.cuh"

namespace {

typedef __nv_bfloat16 bf16;
constexpr int PAGE = 16, TT = 128, MAX_UNITS = 2048;
constexpr int HALF = TT * 128;                     // 128 tokens x 64 latent columns: 16 KB
constexpr int SLOT = 2 * HALF;                     // 128 x 128: 32 KB
constexpr int MAX_SLOTS = 6;
constexpr int THREADS = 256;
constexpr float GROW = 8.0f;                       // log2 units
constexpr float NONE = -1e30f;                     // running maximum of a column that has seen no key

struct LatentParams {
    const int* table;
    int max_pages, num_pages;
    const int* ctx_lens;
    const int* cu;                 // [B + 1] first query token of every sequence; null: sequence b has token b
    int B, H, R, cgs;              // cgs: column groups per sequence
    int q_rows;                    // rows of the query matrix (tokens * H)
    float scale_log2;
    float* part_o;                 // [slots][HG][R]
    float* part_ml;                // [slots][HG][2]
    int* unit_off;                 // for the merge kernel: [MAX_UNITS + 1] tiles before each unit, [MAX_UNITS + 1] pieces
                                   // before each unit, P (0: the tiles are cut as one line)
    int slots_ring;
    int* status;
};

__device__ __forceinline__ float redux_max(float v) {
    float r;
    asm volatile("redux.sync.max.f32 %0, %1, 0xffffffff;" : "=f"(r) : "f"(v));
    return r;
}

// context length that column group cg of sequence b sees
__device__ __forceinline__ int unit_len(const LatentParams& p, int b, int cg, int HG) {
    const int n = p.cu ? p.cu[b + 1] - p.cu[b] : 1;
    if (cg * HG >= n * p.H) return 0;
    const int last = min((cg * HG + HG - 1) / p.H, n - 1);
    return min(p.ctx_lens[b] - n + last + 1, p.max_pages * PAGE);
}

template <int HG>
struct Lay {
    static constexpr int P_BYTES = HG * 256;
    static constexpr int RED = (2 * 4 * HG + 4 * HG + 4 * HG + 4 * HG) * 4;   // maxima (2 parities), own maxima, sums, factors
    static __host__ __device__ int q_bytes(int R) { return HG * R * 2; }
    static __host__ __device__ int fixed(int R) { return q_bytes(R) + P_BYTES + RED + 512 + (MAX_UNITS + 1) * 4 + 1024 + HG * 4; }
};

template <int HG>
__global__ void __launch_bounds__(THREADS, 1)
latent_attn_sm100_kernel(const __grid_constant__ CUtensorMap tmC, const __grid_constant__ CUtensorMap tmQ, const LatentParams p) {
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    const int NS = p.slots_ring, R = p.R, NB = R / 128;        // ring slots; 128-column blocks of a latent
    uint8_t* ring = smem;
    uint8_t* sQ = ring + NS * SLOT;
    uint8_t* sP = sQ + Lay<HG>::q_bytes(R);
    float* red = reinterpret_cast<float*>(sP + Lay<HG>::P_BYTES);    // [2][4][HG]
    float* mown = red + 2 * 4 * HG;                                  // [4][HG] per softmax warp
    float* lred = mown + 4 * HG;                                     // [4][HG]
    float* fown = lred + 4 * HG;                                     // [4][HG]
    int* lim = reinterpret_cast<int*>(fown + 4 * HG);                // [HG] last visible position of every column
    uint64_t* bars = reinterpret_cast<uint64_t*>(lim + HG);
    uint64_t* full = bars;                         // [MAX_SLOTS]
    uint64_t* empty = full + MAX_SLOTS;            // [MAX_SLOTS]
    uint64_t* q_full = empty + MAX_SLOTS;
    uint64_t* q_empty = q_full + 1;
    uint64_t* s_full = q_empty + 1;
    uint64_t* p_ready = s_full + 1;
    uint64_t* o_full = p_ready + 1;
    uint64_t* xch = o_full + 1;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(xch + 1);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
    int* uoff = reinterpret_cast<int*>(reinterpret_cast<uint8_t*>(bars) + 512);   // [units + 1] tiles before each unit
    __shared__ int wsum[THREADS / 32];
    __shared__ int best_p;

    const int warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0), lane = threadIdx.x & 31;   // uniform, and known to be
    if (threadIdx.x == 0) {
        for (int i = 0; i < MAX_SLOTS; ++i) { tc::mbar_init(full + i, 2); tc::mbar_init(empty + i, 1); }
        tc::mbar_init(q_full, 1);
        tc::mbar_init(q_empty, 1);
        tc::mbar_init(s_full, 1);
        tc::mbar_init(p_ready, 4);
        tc::mbar_init(o_full, 1);
        tc::mbar_init(xch, 4);
        *abort_flag = 0;
        tc::fence_barrier_init();
        tc::prefetch_tmap(&tmC);
        tc::prefetch_tmap(&tmQ);
    }
    if (warp == 1) {
        tc::tmem_alloc(tmem_slot, 512);
        tc::tmem_relinquish();
    }
    kb_dep_wait();
    kb_dep_trigger();
    // ---- tiles of every unit and their prefix sums
    const int U = p.B * p.cgs;
    const int per = (U + THREADS - 1) / THREADS;
    {
        int mine = 0;
        for (int i = 0; i < per; ++i) {
            const int u = threadIdx.x * per + i;
            if (u < U) {
                const int t = (unit_len(p, u / p.cgs, u % p.cgs, HG) + TT - 1) / TT;
                uoff[u + 1] = t;
                mine += t;
            }
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
        for (int w = 0; w < warp; ++w) run += wsum[w];
        for (int i = 0; i < per; ++i) {
            const int u = threadIdx.x * per + i;
            if (u < U) {
                run += uoff[u + 1];
                uoff[u + 1] = run;
            }
        }
        if (threadIdx.x == 0) uoff[0] = 0;
    }
    if (threadIdx.x == 0) best_p = 0x7fffffff;
    tc::tc_fence_before();
    __syncthreads();
    tc::tc_fence_after();
    const uint32_t tmem = *tmem_slot;
    const uint32_t tmem_s = tmem, tmem_o = tmem + 64;          // S^T: two buffers of 32 columns; O^T: HG columns per 128-row block
    const uint32_t T = (uint32_t)uoff[U];
    const int g = blockIdx.x;
    int t_begin = 0, t_end = 0, u0 = 0, P = 0;
    if (U <= (int)gridDim.x) {
        // smallest P with sum of ceil(tiles / P) <= CTAs: every warp tries another value
        const int lo = max(1, (int)((T + gridDim.x - 1) / gridDim.x));
        for (int base = lo;; base += THREADS / 32) {
            int n = 0;
            for (int u = lane; u < U; u += 32) n += (uoff[u + 1] - uoff[u] + base + warp - 1) / (base + warp);
            n = __reduce_add_sync(0xffffffffu, n);
            if (lane == 0 && n <= (int)gridDim.x) atomicMin(&best_p, base + warp);
            __syncthreads();
            if (best_p != 0x7fffffff || base > (int)T) break;  // P = T always does: one piece per unit
            __syncthreads();
        }
        P = best_p;
        // this CTA's piece: walk the units' piece counts (every warp for itself, 32 units at a time)
        int run = 0;
        bool found = false;
        for (int ub = 0; ub < U; ub += 32) {
            const int u = ub + lane;
            const int n = u < U ? (uoff[u + 1] - uoff[u] + P - 1) / P : 0;
            int s = n;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int v = __shfl_up_sync(0xffffffffu, s, o);
                if (lane >= o) s += v;
            }
            const int first = run + s - n;                     // pieces before unit u
            if (g == 0 && warp == 0 && u < U) p.unit_off[MAX_UNITS + 1 + u] = first;
            const uint32_t hit = __ballot_sync(0xffffffffu, g >= first && g < first + n);
            if (hit) {
                const int src = __ffs(hit) - 1;
                u0 = ub + src;
                t_begin = uoff[u0] + (g - __shfl_sync(0xffffffffu, first, src)) * P;
                t_end = min(t_begin + P, uoff[u0 + 1]);
                found = true;
            }
            run += __shfl_sync(0xffffffffu, s, 31);
            if (found && g != 0) break;                        // CTA 0 writes all offsets for the merge
        }
        if (g == 0 && warp == 0 && lane == 0) p.unit_off[MAX_UNITS + 1 + U] = run;
    } else {
        // parts of the line: no more than tiles, so that none is empty (the merge walks the parts of a unit)
        const int G = (int)(T < gridDim.x ? T : gridDim.x);
        // (up to 2^24 tiles, in 32 bits: the launcher bounds the context)
        t_begin = g < G ? (int)(T * g / G) : 0;
        t_end = g < G ? (int)(T * (g + 1) / G) : 0;
        if (t_begin < t_end) {
            int hi = U;
            while (hi - u0 > 1) {
                const int m = (u0 + hi) >> 1;
                if (uoff[m] <= t_begin) u0 = m; else hi = m;
            }
        }
    }
    if (g == 0) {
        for (int u = threadIdx.x; u <= U; u += THREADS) p.unit_off[u] = uoff[u];
        if (threadIdx.x == 0) p.unit_off[2 * (MAX_UNITS + 1)] = P;
    }
    // every role walks the same segments: (unit, tiles [a, e) of the unit)
#define FOR_SEGMENTS                                                              \
    for (int u = u0, at = t_begin; at < t_end; at = min(t_end, uoff[u + 1]), ++u) \
        if (uoff[u + 1] > at)

    if (warp == 0 || warp == 6) {
        // ------------------------------------------------------------ TMA: lanes 0-7 each bring one page of this warp's half
        const int pg = lane & 7, hf = warp == 6;
        uint32_t n_slot = 0;
        bool ok = true;
        FOR_SEGMENTS {
            if (!ok) break;
            const int a = at - uoff[u], e = min(t_end, uoff[u + 1]) - uoff[u];
            const int b = u / p.cgs, cg = u % p.cgs;
            const int pages = (unit_len(p, b, cg, HG) + PAGE - 1) / PAGE;
            const int* row = p.table + (long long)b * p.max_pages;
            // pages behind the context repeat the last one: finite numbers that are masked out
            int next = row[min(a * (TT / PAGE) + pg, pages - 1)];
            for (int t = a; t < e && ok; ++t) {
                int page = next;
                if (t + 1 < e) next = row[min((t + 1) * (TT / PAGE) + pg, pages - 1)];
                if (page < 0 || page >= p.num_pages) {
                    atomicMax(p.status, (int)KB_BAD_INDEX);
                    page = 0;
                }
                for (int k = 0; k < NB; ++k, ++n_slot) {
                    const int s = n_slot % NS;
                    if (!tc::mbar_wait(empty + s, ((n_slot / NS) & 1) ^ 1, abort_flag)) { ok = false; break; }
                    if (lane == 0) tc::mbar_expect_tx(full + s, HALF);
                    __syncwarp();
                    if (lane < 8)
                        tc::tma_load_3d(ring + s * SLOT + hf * HALF + pg * PAGE * 128, &tmC, full + s, 0,
                                        (page * (R / 64) + 2 * k + hf) * PAGE, 0);
                }
            }
        }
        if (!ok && lane == 0) {
            atomicMax(p.status, (int)KB_TIMEOUT_TMA);
            const uint64_t t_0 = global_timer_ns();            // copies in flight land before the block can exit
            while (global_timer_ns() - t_0 < 2000000ull) {}
        }
    } else if (warp == 7) {
        // ------------------------------------------------------------ TMA of the queries
        if (lane == 0) {
            uint32_t n_q = 0;
            FOR_SEGMENTS {
                const int b = u / p.cgs, cg = u % p.cgs;
                if (!tc::mbar_wait(q_empty, (n_q & 1) ^ 1, abort_flag)) {
                    atomicMax(p.status, (int)KB_TIMEOUT_TMA);
                    break;
                }
                const int q0 = (p.cu ? p.cu[b] : b) * p.H + cg * HG;
                tc::mbar_expect_tx(q_full, Lay<HG>::q_bytes(R));
                for (int c = 0; c < R / 64; ++c) tc::tma_load_3d(sQ + c * HG * 128, &tmQ, q_full, c * 64, q0, 0);
                ++n_q;
            }
        }
    } else if (warp == 1) {
        // ------------------------------------------------------------ MMA issue
        // The whole warp walks the loop and one elected lane issues: the operands of the products then stay in uniform
        // registers.  (With one thread walking it, moving them there took longer than these small products.)
        const uint32_t id_s = tc::instr_desc_f16(128, HG, 1, 1, 0, 0), id_o = tc::instr_desc_f16(128, HG, 1, 1, 1, 0);
        // descriptors are stepped by adding to their low words: rebuilding them would cost more than the products
        const tc::DescHalves ck = tc::smem_desc_halves(smem_u32(ring), 16, 1024);        // latent tile, K-major
        const tc::DescHalves cm = tc::smem_desc_halves(smem_u32(ring), HALF, 1024);      // latent tile, MN-major
        const tc::DescHalves dq = tc::smem_desc_halves(smem_u32(sQ), 16, 1024), dp = tc::smem_desc_halves(smem_u32(sP), 16, 1024);
        uint32_t n_slot = 0, n_q = 0, n_t = 0;             // n_slot: ring uses before the current tile
        bool ok = true;
        // scores of one 128-column block of a latent tile: eight 16-wide steps, two halves of four
        auto scores = [&](uint32_t s, int k, uint32_t buf) {
            tc::tc_fence_after();
            const uint32_t a_lo = ck.lo + s * (SLOT >> 4), b_lo = dq.lo + k * (2 * HG * 128 >> 4);
            if (tc::elect_one()) {
#pragma unroll
                for (int i = 0; i < 8; ++i)
                    tc::mma_f16_h(tmem_s + buf * 32, a_lo + (((i >> 2) * HALF + (i & 3) * 32) >> 4), ck.hi,
                                  b_lo + (((i >> 2) * HG * 128 + (i & 3) * 32) >> 4), dq.hi, id_s, (k | i) != 0);
            }
            __syncwarp();
        };
        FOR_SEGMENTS {
            if (!ok) break;
            const int a = at - uoff[u], e = min(t_end, uoff[u + 1]) - uoff[u];
            if (!tc::mbar_wait(q_full, n_q & 1, abort_flag)) { ok = false; break; }
            ++n_q;
            int early = 0;                                 // blocks of the current tile whose scores were issued before
            for (int t = a; t < e; ++t, ++n_t) {
                for (int k = early; k < NB; ++k) {
                    const uint32_t n = n_slot + k, s = n % NS;
                    if (!tc::mbar_wait(full + s, (n / NS) & 1, abort_flag)) { ok = false; break; }
                    scores(s, k, n_t & 1);
                }
                if (!ok) break;
                if (tc::elect_one()) {
                    tc::tc_commit(s_full);
                    if (t + 1 == e) tc::tc_commit(q_empty);
                }
                __syncwarp();
                early = 0;
                if (t + 1 < e) {
                    // the next tile's blocks that have arrived in the slots this tile leaves free
                    for (; early < NB && early < NS - NB; ++early) {
                        const uint32_t n = n_slot + NB + early, s = n % NS;
                        if (!__all_sync(0xffffffffu, tc::mbar_try_wait(full + s, (n / NS) & 1))) break;
                        scores(s, early, (n_t + 1) & 1);
                    }
                }
                if (!tc::mbar_wait(p_ready, n_t & 1, abort_flag)) { ok = false; break; }
                tc::tc_fence_after();
                for (int k = 0; k < NB; ++k, ++n_slot) {
                    const uint32_t s = n_slot % NS, a_lo = cm.lo + s * (SLOT >> 4);
                    if (tc::elect_one()) {
#pragma unroll
                        for (int i = 0; i < 8; ++i)        // eight steps of 16 tokens
                            tc::mma_f16_h(tmem_o + k * HG, a_lo + (i * 2048 >> 4), cm.hi,
                                          dp.lo + (((i >> 2) * HG * 128 + (i & 3) * 32) >> 4), dp.hi, id_o, (t > a || i > 0) ? 1u : 0u);
                        tc::tc_commit(empty + s);
                        if (k + 1 == NB && t + 1 == e) tc::tc_commit(o_full);
                    }
                    __syncwarp();
                }
            }
        }
        if (!ok && lane == 0) atomicMax(p.status, (int)KB_TIMEOUT_MMA);
    } else {
        // ------------------------------------------------------------ softmax and output: one token (latent row) per thread
        const int quarter = warp & 3, tk = quarter * 32 + lane;
        const uint32_t lb = (uint32_t)(quarter * 32) << 16;
        float* my_m = mown + quarter * HG;
        float* my_f = fown + quarter * HG;
        uint32_t n_t = 0, n_x = 0, n_seg = 0;
        bool ok = true;
        auto exchange = [&]() -> bool {                        // the four warps have written; bounded, like every wait
            __syncwarp();
            if (lane == 0) tc::mbar_arrive(xch);
            const bool r = tc::mbar_wait(xch, n_x & 1, abort_flag);
            ++n_x;
            return r;
        };
        FOR_SEGMENTS {
            if (!ok) break;
            const int a = at - uoff[u], e = min(t_end, uoff[u + 1]) - uoff[u];
            const int b = u / p.cgs, cg = u % p.cgs;
            const int nq = p.cu ? p.cu[b + 1] - p.cu[b] : 1;
            const int base = p.ctx_lens[b] - nq;
            const int len = unit_len(p, b, cg, HG);
            // columns that are not there see what the last token sees; they are never stored
            if (quarter == 0 && lane < HG) lim[lane] = min(base + min((cg * HG + lane) / p.H, nq - 1), len - 1);
            if (!exchange()) { ok = false; break; }
            float l[HG];
#pragma unroll
            for (int j = 0; j < HG; ++j) l[j] = 0.f;
            float m_col = NONE;                                // lane j (< HG): running maximum of column j
            for (int t = a; t < e; ++t, ++n_t) {
                if (!tc::mbar_wait(s_full, n_t & 1, abort_flag)) { ok = false; break; }
                tc::tc_fence_after();
                float x[HG];
                const uint32_t ts = tmem_s + (n_t & 1) * 32 + lb;
                if constexpr (HG == 32) tc::tmem_ld32(ts, reinterpret_cast<uint32_t*>(x));
                else tc::tmem_ld16(ts, reinterpret_cast<uint32_t*>(x));
                tc::tmem_ld_wait();
                const int pos = t * TT + tk;
                float mine = NONE;
#pragma unroll
                for (int j = 0; j < HG; ++j) {
                    x[j] = pos <= lim[j] ? x[j] * p.scale_log2 : -INFINITY;
                    const float mx = redux_max(x[j]);
                    if (lane == j) mine = fmaxf(mx, NONE);
                }
                float* rb = red + (n_t & 1) * 4 * HG;
                if (lane < HG) rb[quarter * HG + lane] = mine;
                if (!exchange()) { ok = false; break; }
                bool grow = false;
                float f = 1.f;
                if (lane < HG) {
                    const float mx = fmaxf(fmaxf(rb[lane], rb[HG + lane]), fmaxf(rb[2 * HG + lane], rb[3 * HG + lane]));
                    grow = mx > m_col + GROW;
                    if (t == a) {
                        m_col = mx;
                        grow = false;
                    } else if (grow) {
                        f = exp2f(m_col - mx);
                        m_col = mx;
                    }
                    my_m[lane] = m_col;
                    my_f[lane] = f;
                }
                __syncwarp();
                // read in one go: between the stores below every read would wait for the one before
                float mv[HG];
#pragma unroll
                for (int j = 0; j < HG; j += 4) *reinterpret_cast<float4*>(mv + j) = *reinterpret_cast<const float4*>(my_m + j);
                // the four warps see the same maxima and take the same branch; S^T of this tile is complete, so the
                // products into O^T that were issued before it are too
                if (__any_sync(0xffffffffu, grow)) {
#pragma unroll
                    for (int j = 0; j < HG; ++j) l[j] *= my_f[j];
#pragma unroll 1
                    for (int k = 0; k < NB; ++k) {
                        uint32_t o[HG];
                        if constexpr (HG == 32) tc::tmem_ld32(tmem_o + k * HG + lb, o);
                        else tc::tmem_ld16(tmem_o + k * HG + lb, o);
                        tc::tmem_ld_wait();
#pragma unroll
                        for (int j = 0; j < HG; ++j) o[j] = __float_as_uint(__uint_as_float(o[j]) * my_f[j]);
                        if constexpr (HG == 32) tc::tmem_st32(tmem_o + k * HG + lb, o);
                        else tc::tmem_st16(tmem_o + k * HG + lb, o);
                    }
                    tc::tmem_st_wait();
                }
                // P[column][token], K-major with the 128-byte swizzle: 64 tokens per row and half
                uint8_t* prow = sP + (tk >> 6) * HG * 128 + (tk & 7) * 2;
                const int chunk = (tk & 63) >> 3;
#pragma unroll
                for (int j = 0; j < HG; ++j) {
                    const float e2 = exp2f(x[j] - mv[j]);
                    l[j] += e2;
                    *reinterpret_cast<bf16*>(prow + j * 128 + ((chunk ^ (j & 7)) << 4)) = __float2bfloat16(e2);
                }
                tc::fence_proxy_async();
                tc::tc_fence_before();
                __syncwarp();
                if (lane == 0) tc::mbar_arrive(p_ready);
            }
            if (!ok) break;
            // ---- segment output
            float lt = 0.f;
#pragma unroll
            for (int j = 0; j < HG; ++j) {
                const float s = warp_sum(l[j]);
                if (lane == j) lt = s;
            }
            if (lane < HG) lred[quarter * HG + lane] = lt;
            if (!exchange()) { ok = false; break; }
            const long long slot = P ? (long long)g : (long long)g + u;
            if (quarter == 0 && lane < HG) {
                float* ml = p.part_ml + (slot * HG + lane) * 2;
                ml[0] = m_col;
                ml[1] = lred[lane] + lred[HG + lane] + lred[2 * HG + lane] + lred[3 * HG + lane];
            }
            if (!tc::mbar_wait(o_full, n_seg & 1, abort_flag)) { ok = false; break; }
            ++n_seg;
            tc::tc_fence_after();
            const int cols = min(HG, nq * p.H - cg * HG);
            float* po = p.part_o + slot * HG * R + tk;
#pragma unroll 1
            for (int k = 0; k < NB; ++k) {
                uint32_t o[HG];
                if constexpr (HG == 32) tc::tmem_ld32(tmem_o + k * HG + lb, o);
                else tc::tmem_ld16(tmem_o + k * HG + lb, o);
                tc::tmem_ld_wait();
#pragma unroll
                for (int j = 0; j < HG; ++j)
                    if (j < cols) po[(long long)j * R + k * 128] = __uint_as_float(o[j]);
            }
            tc::tc_fence_before();
        }
        if (!ok && lane == 0) atomicMax(p.status, (int)KB_TIMEOUT_EPI);
    }
    tc::tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc::tc_fence_after();
        tc::tmem_dealloc(tmem, 512);
    }
}

// One block per (unit, column): weighs the pieces of the unit and writes the column's latent-space output.
__global__ void __launch_bounds__(128)
latent_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, const int* __restrict__ unit_off,
                    const int* __restrict__ cu, bf16* __restrict__ out, int units, int cgs, int HG, int H, int R, int ctas) {
    kb_dep_trigger();
    kb_dep_wait();
    const int u = blockIdx.x, j = blockIdx.y, b = u / cgs, col = (u % cgs) * HG + j;
    const int q0 = cu ? cu[b] : b, nq = cu ? cu[b + 1] - q0 : 1;
    const int P = unit_off[2 * (MAX_UNITS + 1)];
    const long long T = unit_off[units];
    const int lo = unit_off[u], hi = unit_off[u + 1], first = unit_off[MAX_UNITS + 1 + u];
    if (col >= nq * H) return;
    bf16* dst = out + ((long long)q0 * H + col) * R;
    int s0, n;                                         // first partial of the unit, how many
    if (P) {
        s0 = first;
        n = (hi - lo + P - 1) / P;
    } else {
        const int G = (int)(T < (long long)ctas ? T : (long long)ctas);
        const int g0 = hi > lo ? (int)(((lo + 1ll) * G - 1) / T) : 0;
        s0 = g0 + u;
        n = hi > lo ? (int)(((long long)hi * G - 1) / T) - g0 + 1 : 0;
    }
    const float2* ml = reinterpret_cast<const float2*>(part_ml) + (long long)s0 * HG + j;
    const float* po = part_o + ((long long)s0 * HG + j) * R;
    float M = -INFINITY;
    for (int i = 0; i < n; ++i) M = fmaxf(M, ml[(long long)i * HG].x);
    for (int r = threadIdx.x * 4; r < R; r += 512) {
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
        float den = 0.f;
#pragma unroll 4
        for (int i = 0; i < n; ++i) {
            const float2 x = ml[(long long)i * HG];
            const float4 v = *reinterpret_cast<const float4*>(po + (long long)i * HG * R + r);
            const float w = exp2f(x.x - M);
            den += w * x.y;
            acc.x += w * v.x; acc.y += w * v.y; acc.z += w * v.z; acc.w += w * v.w;
        }
        const float inv = den > 0.f ? 1.0f / den : 0.f;
        const __nv_bfloat162 o0 = __floats2bfloat162_rn(acc.x * inv, acc.y * inv), o1 = __floats2bfloat162_rn(acc.z * inv, acc.w * inv);
        *reinterpret_cast<uint2*>(dst + r) = make_uint2(*reinterpret_cast<const uint32_t*>(&o0), *reinterpret_cast<const uint32_t*>(&o1));
    }
}

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                                  const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                                  CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
int make_tmap(CUtensorMap* m, const void* base, long long cols, long long rows, int box_rows) {
    static EncodeTiledFn enc = nullptr;
    if (!enc) {
        void* ptr = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &q) != cudaSuccess ||
            q != cudaDriverEntryPointSuccess)
            return 100;
        enc = reinterpret_cast<EncodeTiledFn>(ptr);
    }
    cuuint64_t dims[3] = {(cuuint64_t)cols, (cuuint64_t)rows, 1};
    cuuint64_t strides[2] = {(cuuint64_t)cols * 2, (cuuint64_t)rows * cols * 2};
    cuuint32_t box[3] = {64, (cuuint32_t)box_rows, 1};
    cuuint32_t estr[3] = {1, 1, 1};
    const CUresult r = enc(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr,
                           CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                           CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    return r == CUDA_SUCCESS ? 0 : 200 + (int)r;
}

template <int HG>
int ring_slots(int R) {
    int n = (226 * 1024 - Lay<HG>::fixed(R)) / SLOT;      // 1 KB stays for static shared memory
    return n > MAX_SLOTS ? MAX_SLOTS : n;
}

template <int HG>
int launch(const void* q, const void* pages, const LatentParams& p0, bf16* out, int grid, cudaStream_t st) {
    LatentParams p = p0;
    p.slots_ring = ring_slots<HG>(p.R);
    if (p.slots_ring < p.R / 128) return 12;
    static bool flags[64] = {};
    bool* set = kb_device_flag(flags);
    if (!set) return 7;
    if (!*set) {
        if (cudaFuncSetAttribute(latent_attn_sm100_kernel<HG>, cudaFuncAttributeMaxDynamicSharedMemorySize, 226 * 1024) != cudaSuccess)
            return 7;
        *set = true;
    }
    CUtensorMap tmC, tmQ;
    int r = make_tmap(&tmC, pages, 64, (long long)p.num_pages * (p.R / 64) * PAGE, PAGE);
    if (r) return r;
    r = make_tmap(&tmQ, q, p.R, p.q_rows, HG);
    if (r) return r;
    const size_t smem = (size_t)p.slots_ring * SLOT + Lay<HG>::fixed(p.R);
    r = kb_launch_dep(latent_attn_sm100_kernel<HG>, dim3(grid), dim3(THREADS), smem, st, tmC, tmQ, p);
    if (r) return r;
    return kb_launch_dep(latent_merge_kernel, dim3(p.B * p.cgs, HG), dim3(128), 0, st, (const float*)p.part_o, (const float*)p.part_ml,
                         (const int*)p.unit_off, p.cu, out, p.B * p.cgs, p.cgs, HG, p.H, p.R, grid);
}

int sm_count() {
    int sms = 0, dev = 0;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    return sms;
}

}  // namespace

// Query columns per unit for sequences of at most `max_q` new tokens and H heads.
KB_API int kb_latent_cols(int max_q, int H) { return (long long)max_q * H <= 16 ? 16 : 32; }
// Partials that kb_latent_attn may write: floats needed for part_o = slots * cols * R, part_ml = slots * cols * 2.
KB_API int kb_latent_partials(int B, int max_q, int H) {
    const int hg = kb_latent_cols(max_q, H);
    return sm_count() + B * (int)(((long long)max_q * H + hg - 1) / hg);
}
// Whether the kernel covers this latent size (a multiple of 128) and this many units.
KB_API int kb_latent_ok(int B, int max_q, int H, int R) {
    const int hg = kb_latent_cols(max_q, H);
    const long long units = (long long)B * (((long long)max_q * H + hg - 1) / hg);
    if (R < 128 || R % 128 || units > MAX_UNITS) return 0;
    return (hg == 16 ? ring_slots<16>(R) : ring_slots<32>(R)) >= R / 128;
}
// q, out: [tokens, H, R] bf16; pages: [num_pages, R / 64, 16, 64] bf16; unit_off: workspace of 2 * MAX_UNITS + 3 ints.
KB_API int kb_latent_attn(const void* q, const void* pages, const int* table, int max_pages, int num_pages, const int* ctx_lens,
                          const int* cu, int B, int max_q, int tokens, int H, int R, float scale, float* part_o, float* part_ml,
                          int* unit_off, void* out, int* status, cudaStream_t st) {
    if (B < 1 || max_q < 1 || H < 1 || tokens < 1 || max_pages < 1 || num_pages < 1) return 5;
    if (!kb_latent_ok(B, max_q, H, R)) return 12;
    if (((uintptr_t)q & 15) || ((uintptr_t)pages & 15) || ((uintptr_t)out & 15) || ((uintptr_t)part_o & 15)) return 6;
    const int hg = kb_latent_cols(max_q, H);
    LatentParams p;
    p.table = table; p.max_pages = max_pages; p.num_pages = num_pages; p.ctx_lens = ctx_lens; p.cu = cu;
    p.B = B; p.H = H; p.R = R;
    p.cgs = (int)(((long long)max_q * H + hg - 1) / hg);
    p.q_rows = tokens * H;
    p.scale_log2 = scale * 1.4426950408889634f;
    p.part_o = part_o; p.part_ml = part_ml; p.unit_off = unit_off;
    p.slots_ring = 0;
    p.status = status;
    if ((long long)B * p.cgs * ((max_pages + 7) / 8) > (1 << 24)) return 12;
    const int grid = sm_count();
    return hg == 16 ? launch<16>(q, pages, p, (bf16*)out, grid, st) : launch<32>(q, pages, p, (bf16*)out, grid, st);
}
