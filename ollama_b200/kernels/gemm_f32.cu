// 32-bit matrix product of models that run in full precision: D[M, N] (+)= act(A[M, K] . B[N, K]^T), fp32 operands and fp32
// fused multiply-adds (no reduced-precision matrix mode).  64 x 64 tiles, 4 x 4 outputs per thread, two shared-memory stages.
#include "rows.cuh"

namespace {

constexpr int TM = 64, TN = 64, TK = 16, LD = TM + 4;

struct GemmF32Params {
    const float* a;
    const float* b;
    int m, n, k, lda, ldb;
    float* out;
    int ldo, act, accumulate;
};

__global__ void __launch_bounds__(256) gemm_f32_kernel(const __grid_constant__ GemmF32Params p) {
    __shared__ __align__(16) float sa[2][TK][LD], sb[2][TK][LD];
    const int tid = threadIdx.x, m0 = blockIdx.y * TM, n0 = blockIdx.x * TN;
    const int lr = tid >> 2, lk = (tid & 3) * 4;            // this thread's row and first K element of a stage
    const int tx = tid & 15, ty = tid >> 4;
    const float* ap = p.a + (size_t)min(m0 + lr, p.m - 1) * p.lda;
    const float* bp = p.b + (size_t)min(n0 + lr, p.n - 1) * p.ldb;
    auto fetch = [&](const float* row, int k0) {
        const int k = k0 + lk;
        return k < p.k ? *(const float4*)(row + k) : make_float4(0.f, 0.f, 0.f, 0.f);
    };
    auto put = [&](float (&s)[TK][LD], const float4& v) {
        s[lk][lr] = v.x; s[lk + 1][lr] = v.y; s[lk + 2][lr] = v.z; s[lk + 3][lr] = v.w;
    };
    float acc[4][4] = {};
    float4 va = fetch(ap, 0), vb = fetch(bp, 0);
    put(sa[0], va);
    put(sb[0], vb);
    __syncthreads();
    const int nk = (p.k + TK - 1) / TK;
    for (int t = 0; t < nk; t++) {
        const int s = t & 1;
        if (t + 1 < nk) {
            va = fetch(ap, (t + 1) * TK);
            vb = fetch(bp, (t + 1) * TK);
        }
#pragma unroll
        for (int k = 0; k < TK; k++) {
            const float4 x = *(const float4*)&sa[s][k][4 * ty], y = *(const float4*)&sb[s][k][4 * tx];
            const float xv[4] = {x.x, x.y, x.z, x.w}, yv[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(xv[i], yv[j], acc[i][j]);
        }
        if (t + 1 < nk) {
            put(sa[s ^ 1], va);
            put(sb[s ^ 1], vb);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const int row = m0 + 4 * ty + i;
        if (row >= p.m) continue;
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int col = n0 + 4 * tx + j;
            if (col >= p.n) continue;
            float* o = p.out + (size_t)row * p.ldo + col;
            const float v = out_act(acc[i][j], p.act);
            *o = p.accumulate ? *o + v : v;
        }
    }
}

}  // namespace

// k, lda and ldb multiples of four, bases 16-byte aligned.  act: 0 none, 1 square of relu.  Returns a cudaError_t value.
B2_API int b2_gemm_f32(const float* a, int lda, const float* b, int ldb, int m, int n, int k, float* out, int ldo, int act, int accumulate, cudaStream_t st) {
    if (m < 1 || n < 1 || k < 4 || (k & 3) || (lda & 3) || (ldb & 3) || ((uintptr_t)a & 15) || ((uintptr_t)b & 15)) return (int)cudaErrorInvalidValue;
    GemmF32Params p{a, b, m, n, k, lda, ldb, out, ldo, act, accumulate};
    const dim3 grid((n + TN - 1) / TN, (m + TM - 1) / TM);
    if (grid.y > 65535) return (int)cudaErrorInvalidValue;
    gemm_f32_kernel<<<grid, 256, 0, st>>>(p);
    return (int)cudaGetLastError();
}
