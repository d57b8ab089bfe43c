// Gated recurrence whose gates read the current token only, per channel:
//
//   z = sigmoid(z'), c = u + 1/2 where u >= 0, sigmoid(u) below;   S <- (1 - z) S + z c;   out = S silu(g)
//
// The rows hold [z' | u | g], biases added, in 16 or 32 bits; gates, state and results before the last rounding are fp32.  A prompt portion is linear in its state,
// so the warps of a CTA, and the CTAs of a cluster, take consecutive stretches of rows of 32 channels at once: each forms its stretch's decay product and what it
// adds, the state at a stretch's start follows from the ones before it, and a second pass over the values in registers gives the results.  A sequence at position 0
// starts from zero, whatever its slot holds.
#include "rows.cuh"
#include <cooperative_groups.h>

struct GruArgs {
    const void* x;           // [rows][ldx]: z' at column 0, u at off_u, g at off_g
    int ldx, off_u, off_g, width;
    float* state;            // [slots][width]
    const int4* seg;         // portions: first row, rows, slot, position
    const int* slots;        // one-token rows
    const int* positions;
    void* out;               // [rows][ldo]
    int ldo;
};

namespace {

namespace cg = cooperative_groups;
constexpr int STEPS = 16, WARPS = 16, MAX_CLUSTER = 8;

template <bool EXACT>
__device__ __forceinline__ float sig(float v) { return EXACT ? sigmoid_exact(v) : sigmoid_f(v); }

// Weight of the old state and what the token adds.
template <bool EXACT>
__device__ __forceinline__ void gates(float zr, float u, float& keep, float& add) {
    const float z = sig<EXACT>(zr);
    keep = 1.f - z;
    add = z * (u >= 0.f ? u + 0.5f : sig<EXACT>(u));
}

// grid (32-channel groups, CTAs of a cluster, portions)
template <typename T>
__global__ void __launch_bounds__(32 * WARPS) gru_scan_kernel(const __grid_constant__ GruArgs a) {
    constexpr bool EXACT = sizeof(T) == 4;
    __shared__ float s_keep[WARPS][32], s_add[WARPS][32];
    __shared__ float2 s_cta[2][32];                // this CTA's stretch as a whole, of even and odd turns
    const int rank = blockIdx.y, ctas = gridDim.y;
    cg::cluster_group cl = cg::this_cluster();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, ch = blockIdx.x * 32 + lane, c = min(ch, a.width - 1);
    pdl_launch();
    pdl_wait();
    const int4 p = a.seg[blockIdx.z];
    float* st = a.state + (size_t)p.z * a.width + c;
    float state = p.w > 0 ? *st : 0.f;             // at the start of this turn's rows; every thread of every CTA keeps it
    for (int r0 = 0, turn = 0; r0 < p.y; r0 += STEPS * WARPS * ctas, turn ^= 1) {
        const int first = r0 + STEPS * (WARPS * rank + warp);
        const T* x = (const T*)a.x + (size_t)(p.x + first) * a.ldx + c;
        float keep[STEPS], add[STEPS], g[STEPS];
#pragma unroll
        for (int i = 0; i < STEPS; i++) {
            const bool in = first + i < p.y;
            const T* q = x + (size_t)i * a.ldx;
            keep[i] = in ? to_f(q[0]) : 0.f;
            add[i] = in ? to_f(q[a.off_u]) : 0.f;
            g[i] = in ? to_f(q[a.off_g]) : 0.f;
        }
        float k = 1.f, d = 0.f;
#pragma unroll
        for (int i = 0; i < STEPS; i++) {
            gates<EXACT>(keep[i], add[i], keep[i], add[i]);
            if (first + i >= p.y) {
                keep[i] = 1.f;
                add[i] = 0.f;
            }
            k *= keep[i];
            d = fmaf(keep[i], d, add[i]);
        }
        s_keep[warp][lane] = k;
        s_add[warp][lane] = d;
        __syncthreads();
        if (ctas > 1) {
            if (warp == 0) {
                float ck = 1.f, ca = 0.f;
#pragma unroll
                for (int w = 0; w < WARPS; w++) {
                    ck *= s_keep[w][lane];
                    ca = fmaf(s_keep[w][lane], ca, s_add[w][lane]);
                }
                s_cta[turn][lane] = make_float2(ck, ca);
            }
            cl.sync();                             // two sets: nobody writes one before all have passed the turn after its last reading
        }
        float s = state, end = state;              // at this warp's start; at the end of the turn's rows
        for (int q = 0; q < ctas; q++) {
            if (q == rank) {
                s = end;
#pragma unroll
                for (int w = 0; w < WARPS; w++)
                    if (w < warp) s = fmaf(s_keep[w][lane], s, s_add[w][lane]);
            }
            if (ctas > 1) {
                const float2 t = cl.map_shared_rank(s_cta[turn], q)[lane];
                end = fmaf(t.x, end, t.y);
            } else {
#pragma unroll
                for (int w = 0; w < WARPS; w++) end = fmaf(s_keep[w][lane], end, s_add[w][lane]);
            }
        }
        state = end;
        T* o = (T*)a.out + (size_t)(p.x + first) * a.ldo + ch;
#pragma unroll
        for (int i = 0; i < STEPS; i++) {
            s = fmaf(keep[i], s, add[i]);
            if (first + i < p.y && ch < a.width) o[(size_t)i * a.ldo] = from_f<T>(s * g[i] * sig<EXACT>(g[i]));
        }
        __syncthreads();                           // the stretches have been read
    }
    if (ctas > 1) cl.sync();                       // the others have read this CTA's stretch, and the state before it is replaced
    if (rank == 0 && warp == 0 && ch < a.width) *st = state;
}

// grid (channel groups of 256, rows): one token per sequence
template <typename T, bool EXACT>
__global__ void __launch_bounds__(256) gru_step_kernel(const __grid_constant__ GruArgs a) {
    const int c = blockIdx.x * 256 + threadIdx.x, r = blockIdx.y;
    pdl_launch();
    pdl_wait();
    if (c >= a.width) return;
    const T* x = (const T*)a.x + (size_t)r * a.ldx + c;
    float* st = a.state + (size_t)a.slots[r] * a.width + c;
    float keep, add;
    gates<EXACT>(to_f(x[0]), to_f(x[a.off_u]), keep, add);
    const float g = to_f(x[a.off_g]), s = fmaf(keep, a.positions[r] > 0 ? *st : 0.f, add);
    *st = s;
    ((T*)a.out)[(size_t)r * a.ldo + c] = from_f<T>(s * g * sig<EXACT>(g));
}

bool bad(const GruArgs* a) {
    return a->width < 1 || a->off_u < a->width || a->off_g < a->off_u + a->width || a->ldx < a->off_g + a->width || a->ldo < a->width || !a->x || !a->state || !a->out;
}

}  // namespace

// Return a cudaError_t value.  max_rows: rows of the longest portion.
B2_API int b2_gru_scan(const GruArgs* a, int n_seg, int max_rows, int f32, int pdl, cudaStream_t st) {
    if (n_seg < 1 || n_seg > 65535 || max_rows < 1 || !a->seg || bad(a)) return (int)cudaErrorInvalidValue;
    GruArgs c = *a;
    void* args[] = {&c};
    int cluster = 1;
    while (cluster < MAX_CLUSTER && cluster * STEPS * WARPS < max_rows) cluster *= 2;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3((a->width + 31) / 32, cluster, n_seg);
    cfg.blockDim = dim3(32 * WARPS);
    cfg.stream = st;
    cudaLaunchAttribute at[2];
    at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[0].val.programmaticStreamSerializationAllowed = pdl ? 1 : 0;
    at[1].id = cudaLaunchAttributeClusterDimension;
    at[1].val.clusterDim.x = at[1].val.clusterDim.z = 1;
    at[1].val.clusterDim.y = cluster;
    cfg.attrs = at;
    cfg.numAttrs = 2;
    return (int)cudaLaunchKernelExC(&cfg, f32 ? (const void*)gru_scan_kernel<float> : (const void*)gru_scan_kernel<__nv_bfloat16>, args);
}

// exact: the math library's exponentials (32-bit models).
B2_API int b2_gru_step(const GruArgs* a, int rows, int f32, int exact, int pdl, cudaStream_t st) {
    if (rows < 1 || rows > 65535 || !a->slots || !a->positions || bad(a)) return (int)cudaErrorInvalidValue;
    GruArgs c = *a;
    void* args[] = {&c};
    const void* fn = !f32 ? (const void*)gru_step_kernel<__nv_bfloat16, false> : exact ? (const void*)gru_step_kernel<float, true> : (const void*)gru_step_kernel<float, false>;
    return launch_rows(fn, dim3((a->width + 255) / 256, rows), dim3(256), 0, args, st, pdl);
}
