// fp32 matrix product for the 32-bit mode: C[m, n] = sum_k A[m, k] B[n, k] (or B[k, n]) in plain fp32 FMAs.
// Batched, or grouped: the rows of A come in groups (offsets[g] .. offsets[g + 1]), each with its own B.
// 64 x 64 tiles, 256 threads with 4 x 4 results each; any sizes and strides.
#include "common.cuh"

namespace {

constexpr int TM = 64, TN = 64, TK = 16;

struct F32Params {
    const float *A, *B;
    float* C;
    const float* Cin;              // added, may be null; rows ldcin apart (0: one row for all), batches like C
    int M, N, K;
    long long lda, ldb, ldc, ldcin, a_bs, b_bs, c_bs;
    int b_mn;                      // B is [K, N]
    const int* offsets;            // grouped: blockIdx.z is the group, M is ignored
};

__global__ void __launch_bounds__(256) gemm_f32_kernel(const F32Params p) {
    __shared__ float As[TK][TM + 4], Bs[TK][TN + 4];
    kb_dep_trigger();
    kb_dep_wait();
    const int z = blockIdx.z;
    int row0 = blockIdx.y * TM, rows = p.M;
    const float* A = p.A;
    float* C = p.C;
    const float* Cin = p.Cin;
    if (p.offsets) {
        const int lo = p.offsets[z];
        rows = p.offsets[z + 1] - lo;
        A += (long long)lo * p.lda;
        C += (long long)lo * p.ldc;
    } else {
        A += (long long)z * p.a_bs;
        C += (long long)z * p.c_bs;
        if (Cin) Cin += (long long)z * p.c_bs;
    }
    if (row0 >= rows) return;
    const float* B = p.B + (long long)z * p.b_bs;
    const int col0 = blockIdx.x * TN;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < p.K; k0 += TK) {
        for (int i = threadIdx.x; i < TM * TK; i += 256) {
            const int m = i / TK, k = i % TK;
            As[k][m] = row0 + m < rows && k0 + k < p.K ? A[(long long)(row0 + m) * p.lda + k0 + k] : 0.f;
        }
        for (int i = threadIdx.x; i < TN * TK; i += 256) {
            const int n = p.b_mn ? i % TN : i / TK, k = p.b_mn ? i / TN : i % TK;
            float v = 0.f;
            if (col0 + n < p.N && k0 + k < p.K)
                v = p.b_mn ? B[(long long)(k0 + k) * p.ldb + col0 + n] : B[(long long)(col0 + n) * p.ldb + k0 + k];
            Bs[k][n] = v;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < TK; ++k) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) a[i] = As[k][ty * 4 + i];
#pragma unroll
            for (int j = 0; j < 4; ++j) b[j] = Bs[k][tx * 4 + j];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int m = row0 + ty * 4 + i;
        if (m >= rows) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int n = col0 + tx * 4 + j;
            if (n < p.N) C[(long long)m * p.ldc + n] = acc[i][j] + (Cin ? Cin[(long long)m * p.ldcin + n] : 0.f);
        }
    }
}

}  // namespace

// Grouped (offsets not null): `M` is the total number of rows, `batch` the number of groups.
KB_API int kb_gemm_f32(const float* A, const float* B, float* C, const float* Cin, int M, int N, int K, int batch, long long lda,
                       long long ldb, long long ldc, long long ldcin, long long a_bs, long long b_bs, long long c_bs, int b_mn, const int* offsets,
                       cudaStream_t st) {
    if (M < 1 || N < 1 || K < 1 || batch < 1 || batch > 65535 || (M + TM - 1) / TM > 65535) return 5;
    F32Params p{A, B, C, Cin, M, N, K, lda, ldb, ldc, ldcin, a_bs, b_bs, c_bs, b_mn, offsets};
    return kb_launch_dep(gemm_f32_kernel, dim3((N + TN - 1) / TN, (M + TM - 1) / TM, batch), dim3(256), 0, st, p);
}
