// Row-wise operand preparation for matrix products: one or two normalised copies of a row (blocks whose branches normalise
// the same input with weights of their own read it once), two rows side by side, and a column window.  Results are bf16
// (tensor-core operands) or fp32 (32-bit models); columns beyond the row length are written as zeros, so that products may run
// over a padded row length.
//
// The norm is an RMS norm or a layer norm.  Before it, the row itself may be updated in place in the same pass: a branch's result
// under an RMS norm of its own is added, and vectors that join a pass of a loop.
#include "rows.cuh"

struct NormRowsArgs {
    float* x;            // [rows][ldx]; written only when one of y, x0, step is set
    int ldx, k, ldo;     // k values per row; outputs have pitch ldo >= k
    float eps;
    const float* w1;     // [k] weight of the first result
    const float* w2;     // [k] weight of the second result, or null
    void* o1;            // null: only the update
    void* o2;
    int f32;             // element type of the results: 0 bf16, 1 fp32
    const float* b1;     // [k] layer norm: bias of the first result; null: RMS norm
    const float* b2;
    // x += mult * rmsnorm(y) * wy + x0 + step, each term optional
    const float* y;      // [rows][ldy]
    const float* wy;     // [k]
    const float* x0;     // [rows][ldx]
    const float* step;   // [k]
    int ldy;
    float mult;
};

namespace {

// Sum over the CTA of 256; `red` is free again after the call of the next one.
__device__ __forceinline__ float block_sum(float v, float* red) {
    v = warp_sum(v);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.f;
#pragma unroll
    for (int i = 0; i < 8; i++) t += red[i];
    return t;
}

}  // namespace

template <typename T>
__global__ void __launch_bounds__(256) norm_rows_kernel(const __grid_constant__ NormRowsArgs a) {
    __shared__ float red[8];
    const int row = blockIdx.x, tid = threadIdx.x;
    pdl_launch();
    pdl_wait();
    float* x = a.x + (size_t)row * a.ldx;
    if (a.y || a.x0 || a.step) {
        const float* y = a.y ? a.y + (size_t)row * a.ldy : nullptr;
        const float* x0 = a.x0 ? a.x0 + (size_t)row * a.ldx : nullptr;
        float ry = 0.f;
        if (y) {
            float s = 0.f;
            for (int i = tid; i < a.k; i += 256) s += y[i] * y[i];
            ry = a.mult / sqrtf(block_sum(s, red) / (float)a.k + a.eps);
        }
        for (int i = tid; i < a.k; i += 256) {      // a thread reads the same elements again below
            float v = x[i];
            if (y) v += ry * y[i] * a.wy[i];
            if (x0) v += x0[i];
            if (a.step) v += a.step[i];
            x[i] = v;
        }
    }
    if (!a.o1) return;
    float mean = 0.f, ss = 0.f;
    if (a.b1) {
        float s = 0.f;
        for (int i = tid; i < a.k; i += 256) s += x[i];
        mean = block_sum(s, red) / (float)a.k;
    }
    for (int i = tid; i < a.k; i += 256) {
        const float d = x[i] - mean;
        ss += d * d;
    }
    const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)a.k + a.eps);
    T* o1 = (T*)a.o1 + (size_t)row * a.ldo;
    T* o2 = a.o2 ? (T*)a.o2 + (size_t)row * a.ldo : nullptr;
    for (int i = tid; i < a.ldo; i += 256) {
        const bool in = i < a.k;
        const float v = in ? (x[i] - mean) * inv : 0.f;
        o1[i] = from_f<T>(in ? v * a.w1[i] + (a.b1 ? a.b1[i] : 0.f) : 0.f);
        if (o2) o2[i] = from_f<T>(in ? v * a.w2[i] + (a.b2 ? a.b2[i] : 0.f) : 0.f);
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
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    pdl_launch();
    pdl_wait();
    float* x = a.x + (size_t)row * a.ldx;
    float4 v[J], w[J];
#pragma unroll
    for (int j = 0; j < J; j++) {
        const int i = tid + 256 * j;
        v[j] = i < n4 ? *(const float4*)(x + 4 * i) : zero;
        w[j] = i < n4 && a.o1 ? __ldg((const float4*)(a.w1 + 4 * i)) : zero;
    }
    if (a.y || a.x0 || a.step) {
        if (a.y) {
            float4 y[J];
            float s = 0.f;
#pragma unroll
            for (int j = 0; j < J; j++) {
                const int i = tid + 256 * j;
                y[j] = i < n4 ? *(const float4*)(a.y + (size_t)row * a.ldy + 4 * i) : zero;
                s += y[j].x * y[j].x + y[j].y * y[j].y + y[j].z * y[j].z + y[j].w * y[j].w;
            }
            const float ry = a.mult / sqrtf(block_sum(s, red) / (float)a.k + a.eps);
#pragma unroll
            for (int j = 0; j < J; j++) {
                const int i = tid + 256 * j;
                const float4 g = i < n4 ? __ldg((const float4*)(a.wy + 4 * i)) : zero;
                v[j].x += ry * y[j].x * g.x; v[j].y += ry * y[j].y * g.y; v[j].z += ry * y[j].z * g.z; v[j].w += ry * y[j].w * g.w;
            }
        }
#pragma unroll
        for (int j = 0; j < J; j++) {
            const int i = tid + 256 * j;
            if (i >= n4) continue;
            if (a.x0) {
                const float4 u = *(const float4*)(a.x0 + (size_t)row * a.ldx + 4 * i);
                v[j].x += u.x; v[j].y += u.y; v[j].z += u.z; v[j].w += u.w;
            }
            if (a.step) {
                const float4 u = __ldg((const float4*)(a.step + 4 * i));
                v[j].x += u.x; v[j].y += u.y; v[j].z += u.z; v[j].w += u.w;
            }
            *(float4*)(x + 4 * i) = v[j];
        }
    }
    if (!a.o1) return;
    float ss = 0.f;
    if (a.b1) {
        float s = 0.f;
#pragma unroll
        for (int j = 0; j < J; j++) s += v[j].x + v[j].y + v[j].z + v[j].w;
        const float mean = block_sum(s, red) / (float)a.k;
#pragma unroll
        for (int j = 0; j < J; j++) {
            if (tid + 256 * j >= n4) continue;
            v[j].x -= mean; v[j].y -= mean; v[j].z -= mean; v[j].w -= mean;
        }
    }
#pragma unroll
    for (int j = 0; j < J; j++) ss += v[j].x * v[j].x + v[j].y * v[j].y + v[j].z * v[j].z + v[j].w * v[j].w;
    const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)a.k + a.eps);
    T* o1 = (T*)a.o1 + (size_t)row * a.ldo;
    T* o2 = a.o2 ? (T*)a.o2 + (size_t)row * a.ldo : nullptr;
    auto bias = [&](const float* b, int i) { return b ? __ldg((const float4*)(b + 4 * i)) : zero; };
#pragma unroll
    for (int j = 0; j < J; j++) {
        const int i = tid + 256 * j;
        v[j].x *= inv; v[j].y *= inv; v[j].z *= inv; v[j].w *= inv;
        if (i >= n4) continue;
        const float4 b = bias(a.b1, i);
        put4(o1 + 4 * i, v[j].x * w[j].x + b.x, v[j].y * w[j].y + b.y, v[j].z * w[j].z + b.z, v[j].w * w[j].w + b.w);
        if (o2) {
            const float4 u = __ldg((const float4*)(a.w2 + 4 * i)), c = bias(a.b2, i);
            put4(o2 + 4 * i, v[j].x * u.x + c.x, v[j].y * u.y + c.y, v[j].z * u.z + c.z, v[j].w * u.w + c.w);
        }
    }
    for (int i = a.k + tid; i < a.ldo; i += 256) {
        o1[i] = from_f<T>(0.f);
        if (o2) o2[i] = from_f<T>(0.f);
    }
}

B2_API int b2_norm_rows(const NormRowsArgs* a, int rows, int pdl, cudaStream_t st) {
    if (rows < 1 || a->k < 1 || !a->x || (a->ldx & 3) || (a->o1 && (!a->w1 || a->ldo < a->k)) || (a->o2 && (!a->w2 || !a->o1 || !a->b1 != !a->b2)) || (a->y && !a->wy) ||
        (!a->o1 && !a->y && !a->x0 && !a->step))
        return (int)cudaErrorInvalidValue;
    NormRowsArgs c = *a;
    void* args[] = {&c};
    const uintptr_t all = (uintptr_t)a->x | (uintptr_t)a->w1 | (uintptr_t)a->w2 | (uintptr_t)a->o1 | (uintptr_t)a->o2 | (uintptr_t)a->b1 | (uintptr_t)a->b2 |
                          (uintptr_t)a->y | (uintptr_t)a->wy | (uintptr_t)a->x0 | (uintptr_t)a->step;
    if ((a->k & 3) == 0 && a->k <= 4096 && (a->ldo & 3) == 0 && (a->ldy & 3) == 0 && !(all & 15))
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
