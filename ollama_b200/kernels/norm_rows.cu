// Row-wise operand preparation for matrix products: one or two normalised copies of a row (blocks whose branches normalise
// the same input with weights of their own read it once), two rows side by side, and a column window.  Results are bf16
// (tensor-core operands) or fp32 (32-bit models); columns beyond the row length are written as zeros, so that products may run
// over a padded row length.
#include "rows.cuh"

struct NormRowsArgs {
    const float* x;      // [rows][ldx]
    int ldx, k, ldo;     // k values per row; outputs have pitch ldo >= k
    float eps;
    const float* w1;     // [k] weight of the first result
    const float* w2;     // [k] weight of the second result, or null
    void* o1;
    void* o2;
    int f32;             // element type of the results: 0 bf16, 1 fp32
};

template <typename T>
__global__ void __launch_bounds__(256) norm_rows_kernel(const __grid_constant__ NormRowsArgs a) {
    __shared__ float red[8];
    const int row = blockIdx.x, tid = threadIdx.x;
    pdl_launch();
    pdl_wait();
    const float* x = a.x + (size_t)row * a.ldx;
    float ss = 0.f;
    if ((a.k & 3) == 0) {
        for (int i = 4 * tid; i < a.k; i += 1024) {
            const float4 v = *(const float4*)(x + i);
            ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
    } else {
        for (int i = tid; i < a.k; i += 256) ss += x[i] * x[i];
    }
    ss = warp_sum(ss);
    if ((tid & 31) == 0) red[tid >> 5] = ss;
    __syncthreads();
    float t = 0.f;
#pragma unroll
    for (int i = 0; i < 8; i++) t += red[i];
    const float inv = 1.f / sqrtf(t / (float)a.k + a.eps);
    T* o1 = (T*)a.o1 + (size_t)row * a.ldo;
    T* o2 = a.o2 ? (T*)a.o2 + (size_t)row * a.ldo : nullptr;
    for (int i = tid; i < a.ldo; i += 256) {
        const float v = i < a.k ? x[i] * inv : 0.f;
        o1[i] = from_f<T>(i < a.k ? v * a.w1[i] : 0.f);
        if (o2) o2[i] = from_f<T>(i < a.k ? v * a.w2[i] : 0.f);
    }
}

B2_API int b2_norm_rows(const NormRowsArgs* a, int rows, int pdl, cudaStream_t st) {
    if (rows < 1 || a->k < 1 || a->ldo < a->k || (a->ldx & 3) || !a->w1 || (a->o2 && !a->w2)) return (int)cudaErrorInvalidValue;
    NormRowsArgs c = *a;
    void* args[] = {&c};
    return launch_rows(a->f32 ? (const void*)norm_rows_kernel<float> : (const void*)norm_rows_kernel<__nv_bfloat16>, dim3(rows), dim3(256), 0, args, st, pdl);
}

struct JoinRowsArgs {
    const float* a;      // [rows][lda], n_a columns taken
    const float* b;      // [rows][ldb] or null, n_b columns taken
    int lda, n_a, ldb, n_b;
    void* out;           // [rows][ldo]: a at column 0, b at column off_b, zeros elsewhere
    int ldo, off_b, f32;
};

template <typename T>
__global__ void __launch_bounds__(256) join_rows_kernel(const __grid_constant__ JoinRowsArgs p) {
    const int row = blockIdx.x;
    pdl_launch();
    pdl_wait();
    T* o = (T*)p.out + (size_t)row * p.ldo;
    for (int i = threadIdx.x; i < p.ldo; i += 256) {
        float v = 0.f;
        if (i < p.n_a) v = p.a[(size_t)row * p.lda + i];
        else if (p.b && i >= p.off_b && i < p.off_b + p.n_b) v = p.b[(size_t)row * p.ldb + i - p.off_b];
        o[i] = from_f<T>(v);
    }
}

B2_API int b2_join_rows(const JoinRowsArgs* a, int rows, int pdl, cudaStream_t st) {
    if (rows < 1 || a->n_a < 0 || a->n_a > a->ldo || (a->b && (a->off_b < a->n_a || a->off_b + a->n_b > a->ldo))) return (int)cudaErrorInvalidValue;
    JoinRowsArgs c = *a;
    void* args[] = {&c};
    return launch_rows(a->f32 ? (const void*)join_rows_kernel<float> : (const void*)join_rows_kernel<__nv_bfloat16>, dim3(rows), dim3(256), 0, args, st, pdl);
}
