// Grouped GEMM for mixtures of experts:  C[rows of group g] = act(A[rows of group g] x W[g]^T), bf16.
// The rows of A are sorted by group (offsets[g] .. offsets[g + 1], device memory: the host does not know them); the
// weights of the groups are stacked, [G, N, K].  One launch covers all groups.
//
//   TMA (128-byte swizzle) -> shared-memory ring -> tcgen05.mma (128 x BN x 16, fp32 accumulators in tensor
//   memory, two buffers) -> epilogue with the activation, overlapping the next tile's main loop
//
// Every CTA derives the tile list from the offsets: a group with n rows has ceil(n / AM) x ceil(N / BN) tiles.  Tiles
// start at the group's own first row, so the rows are not padded: a tile's operand may run into the next group's rows,
// whose products are not stored.  AM is 128 for prompts and 32 for decoding, where a group has a handful of rows and
// the launch is a stream of weights: the A slot then holds 32 rows (the MMA reads on into whatever lies behind them,
// and those products land in accumulator rows that nobody reads), which leaves the ring to the weights.
// Roles (192 threads): warp 0 = TMA producer, warp 1 = MMA issuer and TMEM owner, warps 2-5 = epilogue.
// All waits are bounded (status word on timeout).
#include <cuda.h>

#include "act.cuh"
#include "tc.cuh"

namespace {

constexpr int BM = 128, BK = 64, MAX_GROUPS = 1024;
template <int BN, int AM> struct Cfg {
    static constexpr int A_STAGE = AM * BK * 2, B_STAGE = BN * BK * 2;
    static constexpr int STAGES = (196 * 1024) / (A_STAGE + B_STAGE) > 8 ? 8 : (196 * 1024) / (A_STAGE + B_STAGE);
    static constexpr int RING = STAGES * (A_STAGE + B_STAGE);
    static constexpr int SLACK = (BM - AM) * BK * 2;     // the 128-row read of the last A slot
    static constexpr int SMEM = RING + SLACK + 1024 + 256 + (MAX_GROUPS + 1) * 4;
    static_assert(SMEM <= 227 * 1024, "shared memory");
};

struct GroupedParams {
    const int* offsets;            // [G + 1]
    int G, N, K, rows, act;        // act: 0 none, 1 exact GELU, 2 squared ReLU
    __nv_bfloat16* C;
    long long ldc;
    int* status;
};

template <int BN, int AM>
__global__ void __launch_bounds__(192, 1)
gemm_grouped_kernel(const __grid_constant__ CUtensorMap tmA, const __grid_constant__ CUtensorMap tmB, const GroupedParams p) {
    using C_ = Cfg<BN, AM>;
    constexpr int STAGES = C_::STAGES, A_STAGE = C_::A_STAGE, B_STAGE = C_::B_STAGE;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    uint8_t* sB = smem;
    uint8_t* sA = smem + STAGES * B_STAGE;
    uint64_t* bars = reinterpret_cast<uint64_t*>(smem + C_::RING + C_::SLACK);
    uint64_t* full = bars;                       // [STAGES] TMA -> MMA
    uint64_t* empty = full + STAGES;             // [STAGES] MMA -> TMA
    uint64_t* acc_full = empty + STAGES;         // [2] MMA -> epilogue
    uint64_t* acc_empty = acc_full + 2;          // [2] epilogue -> MMA
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(acc_empty + 2);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
    int* tile_off = reinterpret_cast<int*>(smem + C_::RING + C_::SLACK + 256);   // [G + 1] row tiles before each group

    const int warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0), lane = threadIdx.x & 31;   // uniform, and known to be
    if (threadIdx.x == 0) {
        for (int s = 0; s < STAGES; ++s) {
            tc::mbar_init(&full[s], 1);
            tc::mbar_init(&empty[s], 1);
        }
        for (int b = 0; b < 2; ++b) {
            tc::mbar_init(&acc_full[b], 1);
            tc::mbar_init(&acc_empty[b], 4);
        }
        *abort_flag = 0;
        tc::fence_barrier_init();
        tc::prefetch_tmap(&tmA);
        tc::prefetch_tmap(&tmB);
    }
    if (warp == 1) {
        tc::tmem_alloc(tmem_slot, 2 * BN);
        tc::tmem_relinquish();
    }
    kb_dep_wait();
    kb_dep_trigger();
    if (warp == 0) {                             // prefix sum of the groups' row tiles
        int run = 0;
        for (int g0 = 0; g0 < p.G; g0 += 32) {
            const int g = g0 + lane;
            int n = 0;
            if (g < p.G) n = (min(p.offsets[g + 1], p.rows) - min(p.offsets[g], p.rows) + AM - 1) / AM;
            n = n < 0 ? 0 : n;
            int s = n;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int v = __shfl_up_sync(0xffffffffu, s, o);
                if (lane >= o) s += v;
            }
            if (g < p.G) tile_off[g] = run + s - n;
            run += __shfl_sync(0xffffffffu, s, 31);
        }
        if (lane == 0) tile_off[p.G] = run;
    }
    tc::tc_fence_before();
    __syncthreads();
    tc::tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    const int tiles_n = (p.N + BN - 1) / BN;
    const int num_tiles = tile_off[p.G] * tiles_n;
    const int kblocks = (p.K + BK - 1) / BK;
    // tile -> group, first row, valid rows, column tile; row tiles of one column tile are neighbours (they share weights)
    auto locate = [&](int tile, int& g, int& row0, int& valid, int& tn) {
        int lo = 0, hi = p.G;
        while (hi - lo > 1) {
            const int m = (lo + hi) >> 1;
            if (tile_off[m] * tiles_n <= tile) lo = m; else hi = m;
        }
        g = lo;                                  // groups without rows have no tiles: the search ends behind them
        const int mt = tile_off[g + 1] - tile_off[g], t = tile - tile_off[g] * tiles_n;
        tn = t / mt;
        row0 = p.offsets[g] + (t % mt) * AM;
        valid = min(AM, min(p.offsets[g + 1], p.rows) - row0);
    };

    if (warp == 0) {
        if (lane == 0) {
            int stage = 0, issued = 0;
            uint32_t phase = 0;
            bool ok = true;
            for (int tile = blockIdx.x; tile < num_tiles && ok; tile += gridDim.x) {
                int g, row0, valid, tn;
                locate(tile, g, row0, valid, tn);
                for (int kb = 0; kb < kblocks; ++kb) {
                    if (!tc::mbar_wait(&empty[stage], phase ^ 1, abort_flag)) {
                        atomicMax(p.status, (int)KB_TIMEOUT_TMA);
                        ok = false;
                        break;
                    }
                    tc::mbar_expect_tx(&full[stage], A_STAGE + B_STAGE);
                    tc::tma_load_3d(sB + stage * B_STAGE, &tmB, &full[stage], kb * BK, tn * BN, g);
                    tc::tma_load_3d(sA + stage * A_STAGE, &tmA, &full[stage], kb * BK, row0, 0);
                    ++issued;
                    if (++stage == STAGES) { stage = 0; phase ^= 1; }
                }
            }
            if (!ok) {                           // let copies already in flight land before the block can exit
                const int inflight = issued < STAGES ? issued : STAGES;
                for (int i = 0; i < inflight; ++i) {
                    int s = stage - 1 - i;
                    uint32_t ph = phase;
                    if (s < 0) { s += STAGES; ph ^= 1; }
                    const uint64_t t0 = global_timer_ns();
                    while (!tc::mbar_try_wait(&full[s], ph) && global_timer_ns() - t0 < 2000000ull) {}
                }
            }
        }
    } else if (warp == 1) {
        // the whole warp walks the loop, one elected lane issues: the operands stay in uniform registers
        const uint32_t idesc = tc::instr_desc_f16(BM, BN, 1, 1, 0, 0);
        const tc::DescHalves da = tc::smem_desc_halves(smem_u32(sA), 16, 1024), db = tc::smem_desc_halves(smem_u32(sB), 16, 1024);
        int stage = 0, it = 0;
        uint32_t phase = 0;
        bool ok = true;
        for (int tile = blockIdx.x; tile < num_tiles && ok; tile += gridDim.x, ++it) {
            const int buf = it & 1;
            if (!tc::mbar_wait(&acc_empty[buf], ((it >> 1) & 1) ^ 1, abort_flag)) { ok = false; break; }
            tc::tc_fence_after();
            for (int kb = 0; kb < kblocks; ++kb) {
                if (!tc::mbar_wait(&full[stage], phase, abort_flag)) { ok = false; break; }
                tc::tc_fence_after();
                const uint32_t a_lo = da.lo + stage * (A_STAGE >> 4), b_lo = db.lo + stage * (B_STAGE >> 4);
                if (tc::elect_one()) {
#pragma unroll
                    for (int k = 0; k < BK / 16; ++k)
                        tc::mma_f16_h(tmem_base + buf * BN, a_lo + (k * 32 >> 4), da.hi, b_lo + (k * 32 >> 4), db.hi, idesc, (kb | k) != 0);
                    tc::tc_commit(&empty[stage]);
                    if (kb + 1 == kblocks) tc::tc_commit(&acc_full[buf]);
                }
                __syncwarp();
                if (++stage == STAGES) { stage = 0; phase ^= 1; }
            }
        }
        if (!ok && lane == 0) atomicMax(p.status, (int)KB_TIMEOUT_MMA);
    } else {
        const int quarter = warp & 3;
        int it = 0;
        for (int tile = blockIdx.x; tile < num_tiles; tile += gridDim.x, ++it) {
            int g, row0, valid, tn;
            locate(tile, g, row0, valid, tn);
            const int buf = it & 1;
            if (!tc::mbar_wait(&acc_full[buf], (it >> 1) & 1, abort_flag)) {
                if (lane == 0) atomicMax(p.status, (int)KB_TIMEOUT_EPI);
                break;
            }
            tc::tc_fence_after();
            const int r = quarter * 32 + lane;
            if (quarter * 32 < valid) {          // uniform over the warp
                const uint32_t taddr = tmem_base + buf * BN + ((uint32_t)(quarter * 32) << 16);
                __nv_bfloat16* dst = p.C + (long long)(row0 + r) * p.ldc;
#pragma unroll 1
                for (int c0 = 0; c0 < BN; c0 += 32) {
                    const int col = tn * BN + c0;
                    if (col >= p.N) break;
                    uint32_t acc[32];
                    tc::tmem_ld32(taddr + c0, acc);
                    tc::tmem_ld_wait();
                    if (r < valid) {
#pragma unroll
                        for (int j = 0; j < 32; j += 8) {
                            float v[8];
#pragma unroll
                            for (int i = 0; i < 8; ++i) {
                                v[i] = __uint_as_float(acc[j + i]);
                                if (p.act == 1) v[i] = gelu_bf16(v[i]);
                                else if (p.act == 2) v[i] = fmaxf(v[i], 0.f) * fmaxf(v[i], 0.f);
                            }
                            if (col + j < p.N) st8(dst + col + j, pack8(v));     // N is a multiple of 8
                        }
                    }
                }
            }
            tc::tc_fence_before();
            __syncwarp();
            if (lane == 0) tc::mbar_arrive(&acc_empty[buf]);
        }
    }
    tc::tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc::tc_fence_after();
        tc::tmem_dealloc(tmem_base, 2 * BN);
    }
}

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                                  const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                                  CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
int make_tmap(CUtensorMap* m, const void* base, long long cols, long long rows, long long ld, long long batch, int box_rows) {
    static EncodeTiledFn enc = nullptr;
    if (!enc) {
        void* ptr = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &q) != cudaSuccess ||
            q != cudaDriverEntryPointSuccess)
            return 100;
        enc = reinterpret_cast<EncodeTiledFn>(ptr);
    }
    cuuint64_t dims[3] = {(cuuint64_t)cols, (cuuint64_t)rows, (cuuint64_t)batch};
    cuuint64_t strides[2] = {(cuuint64_t)ld * 2, (cuuint64_t)rows * ld * 2};
    cuuint32_t box[3] = {BK, (cuuint32_t)box_rows, 1};
    cuuint32_t estr[3] = {1, 1, 1};
    const CUresult r = enc(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr,
                           CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                           CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    return r == CUDA_SUCCESS ? 0 : 200 + (int)r;
}

template <int BN, int AM>
int launch(const void* A, const void* W, const GroupedParams& p, cudaStream_t st) {
    static bool flags[64] = {};
    bool* set = kb_device_flag(flags);
    if (!set) return 7;
    if (!*set) {
        if (cudaFuncSetAttribute(gemm_grouped_kernel<BN, AM>, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg<BN, AM>::SMEM) !=
            cudaSuccess)
            return 7;
        *set = true;
    }
    CUtensorMap tmA, tmB;
    int r = make_tmap(&tmA, A, p.K, p.rows, p.K, 1, AM);
    if (r) return r;
    r = make_tmap(&tmB, W, p.K, p.N, p.K, p.G, BN);
    if (r) return r;
    int sms = 0, dev = 0;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    // most tiles there can be: every group's last row tile may be partial
    const long long most = ((long long)p.rows / AM + (p.G < p.rows ? p.G : p.rows)) * ((p.N + BN - 1) / BN);
    const int grid = (int)(most < sms ? (most < 1 ? 1 : most) : sms);
    return kb_launch_dep(gemm_grouped_kernel<BN, AM>, dim3(grid), dim3(192), (size_t)Cfg<BN, AM>::SMEM, st, tmA, tmB, p);
}

}  // namespace

// A: [rows, K] dense, W: [G, N, K] dense, C: [rows, ldc]; K, N, ldc multiples of 8, 16-byte aligned bases.
// `few`: few rows per group (decode): 32-row tiles.
KB_API int kb_gemm_grouped(const void* A, const void* W, void* C, const int* offsets, int rows, int G, int N, int K, long long ldc,
                           int act, int few, int* status, cudaStream_t st) {
    if (rows < 1 || G < 1 || G > MAX_GROUPS || N < 1 || K < 1 || (N & 7) || (K & 7) || (ldc & 7)) return 5;
    if (((uintptr_t)A & 15) || ((uintptr_t)W & 15) || ((uintptr_t)C & 15)) return 6;
    GroupedParams p{offsets, G, N, K, rows, act, (__nv_bfloat16*)C, ldc, status};
    if (few) return launch<128, 32>(A, W, p, st);
    return launch<256, 128>(A, W, p, st);
}
