// A layer's input of its own per token, for decode steps of one to four rows, sm_100a: one launch, one cluster.
//
//   g = gelu(gate x) * e[token],   y = proj g,   x += mult * y / rms(y) * w   [+ x0] [+ step]
//
// The middle size is small, so the work is latency: the CTAs of a cluster share the rows of both matrices, exchange g and the sums of squares
// through distributed shared memory, and each updates its part of the residual row.  The optional vectors join the next pass of a loop.
#include <cooperative_groups.h>

#include "rows.cuh"

struct SideRowsArgs {
    float* x;                // [nb][ldx], width values
    int ldx, width, k;       // k: padded width, the length of gate's rows (a multiple of 8; x is zero there)
    const void* gate;        // [dim][k]
    const void* e;           // [vocab][lde], this layer's part of a token's row
    int lde, dim, dimp;      // dimp: padded dim, the length of proj's rows (a multiple of 8)
    const int* tokens;       // [nb]
    const void* proj;        // [width][dimp]
    const float* w;          // [width]
    float eps, mult;
    const float* x0;         // [nb][ldx] or null
    const float* step;       // [width] or null
};

namespace {

namespace cg = cooperative_groups;

constexpr int NBM = 4, WARPS = 16;

template <bool F32>
__device__ __forceinline__ float dot8(const void* w, size_t elem, const float* x) {
    float xv[8];
    *(float4*)xv = *(const float4*)x;
    *(float4*)(xv + 4) = *(const float4*)(x + 4);
    float t = 0.f;
    if (F32) {
        const float4 a = __ldg((const float4*)((const float*)w + elem)), b = __ldg((const float4*)((const float*)w + elem) + 1);
        t = a.x * xv[0] + a.y * xv[1] + a.z * xv[2] + a.w * xv[3] + b.x * xv[4] + b.y * xv[5] + b.z * xv[6] + b.w * xv[7];
    } else {
        const uint4 v = __ldg((const uint4*)((const __nv_bfloat16*)w + elem));
        const uint32_t q[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int i = 0; i < 4; i++) t = fmaf(__uint_as_float(q[i] & 0xffff0000u), xv[2 * i + 1], fmaf(__uint_as_float(q[i] << 16), xv[2 * i], t));
    }
    return t;
}

// smem: g [NB][dimp], y [NB][rows of a CTA]
template <bool F32, int NB>
__global__ void __launch_bounds__(32 * WARPS) side_rows_kernel(const __grid_constant__ SideRowsArgs a, int nb) {
    using T = typename std::conditional<F32, float, __nv_bfloat16>::type;
    extern __shared__ __align__(16) float sm[];
    __shared__ float s_ss[NBM];                    // sum of squares of the CTA's part
    __shared__ float s_w[WARPS][NBM];
    cg::cluster_group cl = cg::this_cluster();
    const int cr = cl.block_rank(), cn = cl.num_blocks(), tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int per = (a.width + cn - 1) / cn, r0 = cr * per, r1 = min(r0 + per, a.width);
    float* g = sm;
    float* y = sm + NB * a.dimp;
    const T* gate = (const T*)a.gate;
    const T* proj = (const T*)a.proj;
    constexpr int LINE = 128 / (int)sizeof(T);
    pdl_launch();
    for (int j = cr * WARPS + warp; j < a.dim; j += cn * WARPS)
        for (int c = lane * LINE; c < a.k; c += 32 * LINE) asm volatile("prefetch.global.L2 [%0];" ::"l"(gate + (size_t)j * a.k + c));
    for (size_t c = (size_t)r0 * a.dimp + tid * LINE; r0 < r1 && c < (size_t)r1 * a.dimp; c += 32 * WARPS * LINE) asm volatile("prefetch.global.L2 [%0];" ::"l"(proj + c));
    pdl_wait();
    for (int i = tid; i < NB * (a.dimp - a.dim); i += 32 * WARPS) {
        const int b = i / (a.dimp - a.dim);
        g[b * a.dimp + a.dim + i - b * (a.dimp - a.dim)] = 0.f;
    }
    cl.sync();                                     // every CTA runs before its shared memory is written to
    for (int j = cr * WARPS + warp; j < a.dim; j += cn * WARPS) {
        float acc[NB];
#pragma unroll
        for (int b = 0; b < NB; b++) acc[b] = 0.f;
        for (int c = 8 * lane; c < a.k; c += 256) {
#pragma unroll
            for (int b = 0; b < NB; b++)
                if (b < nb) acc[b] += dot8<F32>(gate, (size_t)j * a.k + c, a.x + (size_t)b * a.ldx + c);
        }
#pragma unroll
        for (int b = 0; b < NB; b++) {
            if (b >= nb) break;
            const float v = gelu_tanh_f(warp_sum(acc[b])) * to_f(((const T*)a.e)[(size_t)a.tokens[b] * a.lde + j]);
            if (lane < cn) cl.map_shared_rank(g, lane)[b * a.dimp + j] = v;
        }
    }
    cl.sync();
    float ss[NB];
#pragma unroll
    for (int b = 0; b < NB; b++) ss[b] = 0.f;
    for (int r = r0 + tid; r < r1; r += 32 * WARPS) {      // rows of proj are short: a thread each
        float acc[NB];
#pragma unroll
        for (int b = 0; b < NB; b++) acc[b] = 0.f;
#pragma unroll 4
        for (int c = 0; c < a.dimp; c += 8) {
#pragma unroll
            for (int b = 0; b < NB; b++)
                if (b < nb) acc[b] += dot8<F32>(proj, (size_t)r * a.dimp + c, g + b * a.dimp + c);
        }
#pragma unroll
        for (int b = 0; b < NB; b++) {
            y[b * per + r - r0] = acc[b];
            ss[b] += acc[b] * acc[b];
        }
    }
#pragma unroll
    for (int b = 0; b < NB; b++) {
        const float s = warp_sum(ss[b]);
        if (lane == 0) s_w[warp][b] = s;
    }
    __syncthreads();
    if (tid < NB) {
        float s = 0.f;
        for (int i = 0; i < WARPS; i++) s += s_w[i][tid];
        s_ss[tid] = s;
    }
    cl.sync();
#pragma unroll
    for (int b = 0; b < NB; b++) {
        if (b >= nb) break;
        float s = lane < cn ? *cl.map_shared_rank(&s_ss[b], lane) : 0.f;
        s = warp_sum(s);
        const float inv = a.mult / sqrtf(s / (float)a.width + a.eps);
        for (int r = r0 + tid; r < r1; r += 32 * WARPS) {
            float* o = a.x + (size_t)b * a.ldx + r;
            float v = *o + inv * y[b * per + r - r0] * a.w[r];
            if (a.x0) v += a.x0[(size_t)b * a.ldx + r];
            if (a.step) v += a.step[r];
            *o = v;
        }
    }
    cl.sync();                                     // nobody leaves while its sums are read
}

template <bool F32, int NB>
int launch(const SideRowsArgs& a, int nb, int cluster, size_t smem, int pdl, cudaStream_t st) {
    static PerDeviceOnce once;
    const void* fn = (const void*)side_rows_kernel<F32, NB>;
    if (once.first()) {
        cudaFuncSetAttribute(fn, cudaFuncAttributeNonPortableClusterSizeAllowed, 1);
        cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024);
    }
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(cluster);
    cfg.blockDim = dim3(32 * WARPS);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute at[2];
    at[0].id = cudaLaunchAttributeClusterDimension;
    at[0].val.clusterDim = {(unsigned)cluster, 1, 1};
    at[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[1].val.programmaticStreamSerializationAllowed = pdl ? 1 : 0;
    cfg.attrs = at;
    cfg.numAttrs = 2;
    SideRowsArgs c = a;
    void* args[] = {&c, &nb};
    return (int)cudaLaunchKernelExC(&cfg, fn, args);
}

}  // namespace

// cudaErrorNotSupported: more rows or sizes than the launch takes, nothing was launched.
B2_API int b2_side_rows(const SideRowsArgs* a, int nb, int f32, int cluster, int pdl, cudaStream_t st) {
    if (nb < 1 || a->width < 1 || a->k < a->width || (a->k & 7) || (a->ldx & 3) || a->dim < 1 || a->dimp < a->dim || (a->dimp & 7) || cluster < 1 || cluster > 16 ||
        ((uintptr_t)a->x & 15) || ((uintptr_t)a->gate & 15) || ((uintptr_t)a->proj & 15))
        return (int)cudaErrorInvalidValue;
    const int m = nb == 1 ? 1 : NBM;
    const size_t smem = ((size_t)m * a->dimp + (size_t)m * ((a->width + cluster - 1) / cluster)) * 4;
    if (nb > NBM || smem > 160 * 1024) return (int)cudaErrorNotSupported;
    if (f32) return m == 1 ? launch<true, 1>(*a, nb, cluster, smem, pdl, st) : launch<true, NBM>(*a, nb, cluster, smem, pdl, st);
    return m == 1 ? launch<false, 1>(*a, nb, cluster, smem, pdl, st) : launch<false, NBM>(*a, nb, cluster, smem, pdl, st);
}
