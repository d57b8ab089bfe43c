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

template <typename T>
__device__ __forceinline__ void put4(T* o, float a, float b, float c, float d) {
    if (sizeof(T) == 2) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
        *(uint2*)o = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
    } else {
        *(float4*)o = make_float4(a, b, c, d);
    }
}

// Rows of up to 4096 values that are a multiple of four: the row stays in registers, all loads of a row are under way together.
template <typename T>
__global__ void __launch_bounds__(256) norm_rows4_kernel(const __grid_constant__ NormRowsArgs a) {
    constexpr int J = 4;
    __shared__ float red[8];
    const int row = blockIdx.x, tid = threadIdx.x, n4 = a.k >> 2;
    pdl_launch();
    pdl_wait();
    const float* x = a.x + (size_t)row * a.ldx;
    float4 v[J], w[J];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < J; j++) {
        const int i = tid + 256 * j;
        v[j] = i < n4 ? *(const float4*)(x + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
        w[j] = i < n4 ? __ldg((const float4*)(a.w1 + 4 * i)) : v[j];
    }
#pragma unroll
    for (int j = 0; j < J; j++) ss += v[j].x * v[j].x + v[j].y * v[j].y + v[j].z * v[j].z + v[j].w * v[j].w;
    ss = warp_sum(ss);
    if ((tid & 31) == 0) red[tid >> 5] = ss;
    __syncthreads();
    float t = 0.f;
#pragma unroll
    for (int i = 0; i < 8; i++) t += red[i];
    const float inv = 1.f / sqrtf(t / (float)a.k + a.eps);
    T* o1 = (T*)a.o1 + (size_t)row * a.ldo;
    T* o2 = a.o2 ? (T*)a.o2 + (size_t)row * a.ldo : nullptr;
#pragma unroll
    for (int j = 0; j < J; j++) {
        const int i = tid + 256 * j;
        v[j].x *= inv; v[j].y *= inv; v[j].z *= inv; v[j].w *= inv;
        if (i < n4) put4(o1 + 4 * i, v[j].x * w[j].x, v[j].y * w[j].y, v[j].z * w[j].z, v[j].w * w[j].w);
    }
    if (o2) {
#pragma unroll
        for (int j = 0; j < J; j++) {
            const int i = tid + 256 * j;
            if (i < n4) {
                const float4 u = __ldg((const float4*)(a.w2 + 4 * i));
                put4(o2 + 4 * i, v[j].x * u.x, v[j].y * u.y, v[j].z * u.z, v[j].w * u.w);
            }
        }
    }
    for (int i = a.k + tid; i < a.ldo; i += 256) {
        o1[i] = from_f<T>(0.f);
        if (o2) o2[i] = from_f<T>(0.f);
    }
}

B2_API int b2_norm_rows(const NormRowsArgs* a, int rows, int pdl, cudaStream_t st) {
    if (rows < 1 || a->k < 1 || a->ldo < a->k || (a->ldx & 3) || !a->w1 || (a->o2 && !a->w2)) return (int)cudaErrorInvalidValue;
    NormRowsArgs c = *a;
    void* args[] = {&c};
    if ((a->k & 3) == 0 && a->k <= 4096 && (a->ldo & 3) == 0 &&
        !(((uintptr_t)a->x | (uintptr_t)a->w1 | (uintptr_t)a->w2 | (uintptr_t)a->o1 | (uintptr_t)a->o2) & 15))
        return launch_rows(a->f32 ? (const void*)norm_rows4_kernel<float> : (const void*)norm_rows4_kernel<__nv_bfloat16>, dim3(rows), dim3(256), 0, args, st, pdl);
    return launch_rows(a->f32 ? (const void*)norm_rows_kernel<float> : (const void*)norm_rows_kernel<__nv_bfloat16>, dim3(rows), dim3(256), 0, args, st, pdl);
}

struct JoinRowsArgs {
    const float* a;      // [rows][lda], n_a columns taken
    const float* b;      // [rows][ldb] or null, n_b columns taken
    int lda, n_a, ldb, n_b;
    void* out;           // [rows][ldo]: a at column 0, b at column off_b, zeros elsewhere
    int ldo, off_b, f32;
};

// grid (rows, column blocks of 1024); VEC: every width, pitch and offset is a multiple of four
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) join_rows_kernel(const __grid_constant__ JoinRowsArgs p) {
    const int row = blockIdx.x;
    pdl_launch();
    pdl_wait();
    T* o = (T*)p.out + (size_t)row * p.ldo;
    const int c0 = blockIdx.y * 1024;
    if (VEC) {
        const int i = c0 + 4 * threadIdx.x;
        if (i >= p.ldo) return;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < p.n_a) v = *(const float4*)(p.a + (size_t)row * p.lda + i);
        else if (p.b && i >= p.off_b && i < p.off_b + p.n_b) v = *(const float4*)(p.b + (size_t)row * p.ldb + i - p.off_b);
        put4(o + i, v.x, v.y, v.z, v.w);
        return;
    }
    for (int i = c0 + threadIdx.x; i < min(c0 + 1024, p.ldo); i += 256) {
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
    const bool vec = !((a->n_a | a->n_b | a->lda | a->ldb | a->ldo | a->off_b) & 3) && !(((uintptr_t)a->a | (uintptr_t)a->b | (uintptr_t)a->out) & 15);
    const void* fn = a->f32 ? (vec ? (const void*)join_rows_kernel<float, true> : (const void*)join_rows_kernel<float, false>)
                            : (vec ? (const void*)join_rows_kernel<__nv_bfloat16, true> : (const void*)join_rows_kernel<__nv_bfloat16, false>);
    return launch_rows(fn, dim3(rows, (a->ldo + 1023) / 1024), dim3(256), 0, args, st, pdl);
}
