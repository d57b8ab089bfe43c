// 32-bit matrix product of models that run in full precision: D[M, N] (+)= act(A[M, K] . B[N, K]^T), fp32 operands and fp32
// fused multiply-adds (no reduced-precision matrix mode).  64 x 64 tiles, 4 x 4 outputs per thread, two shared-memory stages.  The epilogues
// are those of the tensor-core product (gemm_tc.cu).
#include "rows.cuh"

namespace {

constexpr int TM = 64, TN = 64, TK = 16, LD = TM + 4;

__global__ void __launch_bounds__(256) gemm_f32_kernel(const __grid_constant__ GemmRowsArgs p) {
    __shared__ __align__(16) float sa[2][TK][LD], sb[2][TK][LD];
    const int tid = threadIdx.x, m0 = blockIdx.y * TM, n0 = blockIdx.x * TN;
    const int lr = tid >> 2, lk = (tid & 3) * 4;            // this thread's row and first K element of a stage
    const int tx = tid & 15, ty = tid >> 4;
    const int e = p.tile_expert ? p.tile_expert[m0 >> 7] : 0;
    if (e < 0) return;
    const float* ap = (const float*)p.a + (size_t)min(m0 + lr, p.m - 1) * p.lda;
    const float* bp = (const float*)p.b + ((size_t)e * p.n + min(n0 + lr, p.n - 1)) * p.ldb;
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
        float v[4];
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int col = min(n0 + 4 * tx + j, p.n - 1);
            v[j] = acc[i][j] + (p.bias ? p.bias[col] : 0.f);
        }
        if (p.act >= GLU_BASE) {
#pragma unroll
            for (int j = 0; j < 4; j += 2) {
                const int col = n0 + 4 * tx + j;
                if (col < p.n) ((float*)p.out)[(size_t)row * p.ldo + (col >> 1)] = glu_act_exact(v[j], v[j + 1], p.act - GLU_BASE, SWIGLU_ALPHA, p.limit);
            }
            continue;
        }
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int col = n0 + 4 * tx + j;
            if (col >= p.n) continue;
            float* o = (float*)p.out + (size_t)row * p.ldo + col;
            float r = out_act<true>(v[j], p.act, p.act_p, p.act_q);
            if (p.mul) r *= ((const float*)p.mul)[(size_t)p.mul_row[row] * p.ldm + col];
            r *= p.alpha;
            *o = p.accumulate ? *o + r : r;
        }
    }
}

}  // namespace

// k, lda and ldb multiples of four, n even for gated products, bases 16-byte aligned.  Returns a cudaError_t value.
B2_API int b2_gemm_rows_f32(const GemmRowsArgs* g, cudaStream_t st) {
    const int glu = g->act >= GLU_BASE ? 1 : 0;
    if (g->m < 1 || g->n < 1 || g->k < 4 || (g->k & 3) || (g->lda & 3) || (g->ldb & 3) || ((uintptr_t)g->a & 15) || ((uintptr_t)g->b & 15) || g->out_type || g->copy || g->tail || g->act < 0 ||
        (!glu && g->act > ACT_LAST) || g->act > GLU_BASE + 2 || (glu && ((g->n & 1) || g->accumulate || g->mul)) || (g->mul && !g->mul_row) ||
        (g->tile_expert && (g->experts < 1 || (g->m & 127))))
        return (int)cudaErrorInvalidValue;
    const dim3 grid((g->n + TN - 1) / TN, (g->m + TM - 1) / TM);
    if (grid.y > 65535) return (int)cudaErrorInvalidValue;
    gemm_f32_kernel<<<grid, 256, 0, st>>>(*g);
    return (int)cudaGetLastError();
}
