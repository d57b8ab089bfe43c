// Weighted sums over the depth of a model, with the layer norm of the next layer: of designs whose layers read a learned average of the embedding output and
// all earlier layers' results.
//
//   x = sum_j w[j] X_j,   h = (x - mean) / sqrt(var + eps) * g + b
//
// X_0 .. X_(n-1) stand one after the other, each a block of the step's rows.  x is written as the start of X_n, which the layer's products add to.  A cluster
// of CTAs shares a row (several when the step has few rows: reading a long history is all there is to do), each with its own columns; the groups of
// threads of a CTA share the history and add their parts up in shared memory.  Mean and squared deviations of the CTAs' columns are formed locally and combined
// (Chan, Golub and LeVeque's pairwise update), so that the cluster meets once.
#include "rows.cuh"
#include <cooperative_groups.h>

struct DepthRowsArgs {
    const float* hist;       // [n][rows][ldx]
    long long stride;        // floats from one block to the next
    const float* w;          // [n]
    int n, k, ldx;           // k values per row, columns up to ldx are zero
    float* x;                // [rows][ldx]
    const float* g;          // [k] norm weight
    const float* b;          // [k]
    void* h;                 // [rows][ldo] bf16 or (f32) fp32, zeros behind k; null: only x
    int ldo, f32;
    float eps;
};

namespace {

namespace cg = cooperative_groups;
constexpr int THREADS = 256, ITEMS = 4, BATCH = 8, MAX_CLUSTER = 8;
constexpr int MAX_COLS = THREADS * ITEMS * 4;      // columns of a CTA

template <typename T>
__device__ __forceinline__ void put4(T* o, const float4& v) {
    if (sizeof(T) == 2) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
        *(uint2*)o = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
    } else {
        *(float4*)o = v;
    }
}

__device__ __forceinline__ float block_sum(float v, float* red) {
    v = warp_sum(v);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.f;
#pragma unroll
    for (int i = 0; i < THREADS / 32; i++) t += red[i];
    return t;
}

// grid (CTAs of a row, rows), clusters of gridDim.x.  cols: columns per CTA, a multiple of four; groups: parts of the history, a power of two with
// cols / 4 <= 256 / groups where it is above 1.
template <typename T>
__global__ void __launch_bounds__(THREADS) depth_rows_kernel(const __grid_constant__ DepthRowsArgs a, int cols, int groups) {
    __shared__ float4 part[THREADS];
    __shared__ float red[THREADS / 32];
    __shared__ float2 stats;                       // mean and squared deviations of this CTA's columns
    const int row = blockIdx.y, tid = threadIdx.x, per = THREADS / groups, grp = tid / per, slot = tid - grp * per;
    const int c0 = blockIdx.x * cols, c1 = min(c0 + cols, a.ldx), items = (c1 - c0) >> 2;
    pdl_launch();
    pdl_wait();
    const float* src = a.hist + (size_t)row * a.ldx + c0;
    float4 v[ITEMS];
#pragma unroll
    for (int i = 0; i < ITEMS; i++) v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < ITEMS; i++) {
        const int it = slot + per * i;
        if (it >= items || (groups > 1 && i > 0)) break;
        for (int j0 = grp; j0 < a.n; j0 += groups * BATCH) {
            float4 y[BATCH];
            float f[BATCH];
#pragma unroll
            for (int u = 0; u < BATCH; u++) {
                const int j = j0 + groups * u;
                const bool in = j < a.n;
                f[u] = in ? __ldg(a.w + j) : 0.f;
                y[u] = in ? *(const float4*)(src + (size_t)j * a.stride + 4 * it) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
#pragma unroll
            for (int u = 0; u < BATCH; u++) {
                v[i].x = fmaf(f[u], y[u].x, v[i].x); v[i].y = fmaf(f[u], y[u].y, v[i].y);
                v[i].z = fmaf(f[u], y[u].z, v[i].z); v[i].w = fmaf(f[u], y[u].w, v[i].w);
            }
        }
    }
    if (groups > 1) {                              // every group ends up with the sum; the first one goes on with it
        part[tid] = v[0];
        __syncthreads();
        v[0] = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int q = 0; q < groups; q++) {
            const float4 y = part[q * per + slot];
            v[0].x += y.x; v[0].y += y.y; v[0].z += y.z; v[0].w += y.w;
        }
    }
    const bool lead = grp == 0;
    float* x = a.x + (size_t)row * a.ldx + c0;
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < ITEMS; i++) {
        const int it = slot + per * i;
        if (!lead || it >= items || (groups > 1 && i > 0)) break;
        *(float4*)(x + 4 * it) = v[i];
        s += v[i].x + v[i].y + v[i].z + v[i].w;    // columns behind k are zero
    }
    if (!a.h) return;
    const int mine = max(0, min(c1, a.k) - c0);    // this CTA's columns of the row
    float mean = block_sum(s, red) / (float)max(mine, 1);
    float m2 = 0.f;
#pragma unroll
    for (int i = 0; i < ITEMS; i++) {
        const int it = slot + per * i;
        if (!lead || it >= items || (groups > 1 && i > 0)) break;
        const float q[4] = {v[i].x, v[i].y, v[i].z, v[i].w};
#pragma unroll
        for (int e = 0; e < 4; e++)
            if (4 * it + e < mine) m2 += (q[e] - mean) * (q[e] - mean);
    }
    m2 = block_sum(m2, red);
    if (gridDim.x > 1) {
        cg::cluster_group cl = cg::this_cluster();
        if (tid == 0) stats = make_float2(mean, m2);
        cl.sync();
        float n = 0.f, mn = 0.f, sq = 0.f;
        for (int r = 0; r < (int)gridDim.x; r++) {
            const float2 o = *cl.map_shared_rank(&stats, r);
            const float cnt = (float)max(0, min(min((r + 1) * cols, a.ldx), a.k) - r * cols);
            if (cnt == 0.f) continue;
            const float d = o.x - mn, all = n + cnt;
            sq += o.y + d * d * n * cnt / all;
            mn += d * cnt / all;
            n = all;
        }
        mean = mn;
        m2 = sq;
        cl.sync();                                 // nobody leaves while its numbers are read
    }
    const float inv = 1.f / sqrtf(m2 / (float)a.k + a.eps);
    T* o = (T*)a.h + (size_t)row * a.ldo + c0;
#pragma unroll
    for (int i = 0; i < ITEMS; i++) {
        const int it = slot + per * i;
        if (!lead || it >= items || (groups > 1 && i > 0)) break;
        float q[4] = {v[i].x, v[i].y, v[i].z, v[i].w};
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int c = c0 + 4 * it + e;
            q[e] = c < a.k ? (q[e] - mean) * inv * __ldg(a.g + c) + __ldg(a.b + c) : 0.f;
        }
        put4(o + 4 * it, make_float4(q[0], q[1], q[2], q[3]));
    }
}

}  // namespace

// ldx = ldo, a multiple of four up to 32768.  Returns a cudaError_t value.
B2_API int b2_depth_rows(const DepthRowsArgs* a, int rows, int pdl, cudaStream_t st) {
    if (rows < 1 || rows > 65535 || a->n < 1 || a->k < 1 || a->k > a->ldx || (a->ldx & 3) || (a->stride & 3) || !a->hist || !a->w || !a->x || (a->h && (!a->g || !a->b || a->ldo != a->ldx)) ||
        (((uintptr_t)a->hist | (uintptr_t)a->x | (uintptr_t)a->h) & 15))
        return (int)cudaErrorInvalidValue;
    if (a->ldx > MAX_COLS * MAX_CLUSTER) return (int)cudaErrorNotSupported;
    int cluster = 1;
    while (cluster < MAX_CLUSTER && (a->ldx > MAX_COLS * cluster || (rows * cluster < 64 && a->ldx >= 256 * cluster))) cluster *= 2;
    const int cols = ((a->ldx + cluster - 1) / cluster + 3) & ~3;
    int groups = 1;
    while (groups < 8 && cols / 4 <= THREADS / (2 * groups) && groups * BATCH < a->n) groups *= 2;
    DepthRowsArgs c = *a;
    int cc = cols, gg = groups;
    void* args[] = {&c, &cc, &gg};
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(cluster, rows);
    cfg.blockDim = dim3(THREADS);
    cfg.stream = st;
    cudaLaunchAttribute at[2];
    at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[0].val.programmaticStreamSerializationAllowed = pdl ? 1 : 0;
    at[1].id = cudaLaunchAttributeClusterDimension;
    at[1].val.clusterDim.x = cluster;
    at[1].val.clusterDim.y = at[1].val.clusterDim.z = 1;
    cfg.attrs = at;
    cfg.numAttrs = 2;
    return (int)cudaLaunchKernelExC(&cfg, a->f32 ? (const void*)depth_rows_kernel<float> : (const void*)depth_rows_kernel<__nv_bfloat16>, args);
}
