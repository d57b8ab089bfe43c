// Gated recurrence whose gates read the current token only, per channel:
//
//   z = sigmoid(z'), c = u + 1/2 where u >= 0, sigmoid(u) below;   S <- (1 - z) S + z c;   out = S silu(g)
//
// The rows hold [z' | u | g], biases added, in 16 or 32 bits; gates, state and results before the last rounding are fp32.  A prompt portion is linear in its state,
// so the warps of a CTA, and the CTAs of a cluster, take consecutive stretches of rows of 64 channels at once: each forms its stretch's decay product and what it
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
constexpr int STEPS = 8, WARPS = 16, MAX_CLUSTER = 8;

template <bool EXACT>
__device__ __forceinline__ float sig(float v) { return EXACT ? sigmoid_exact(v) : sigmoid_f(v); }

// Weight of the old state, what the token adds, and the output gate silu(g).  The three sigmoids share one reciprocal (of a product that stays below 2^126, for exponents
// beyond which a sigmoid is below 3e-13): the special-function unit is what bounds the scan.
__device__ __forceinline__ void gates3(float zr, float u, float g, float& keep, float& add, float& gate) {
    constexpr float LAST = 29.f;
    const float dz = 1.f + __expf(fminf(-zr, LAST)), dg = 1.f + __expf(fminf(-g, LAST)), du = 1.f + __expf(u < 0.f ? fminf(-u, LAST) : -LAST);
    const float zg = dz * dg, r = __fdividef(1.f, zg * du), ru = r * zg, rzg = r * du;
    const float z = rzg * dg;
    keep = 1.f - z;
    add = z * (u >= 0.f ? u + 0.5f : ru);
    gate = g * (rzg * dz);
}

// Weight of the old state and what the token adds.
template <bool EXACT>
__device__ __forceinline__ void gates(float zr, float u, float& keep, float& add) {
    const float z = sig<EXACT>(zr);
    keep = 1.f - z;
    add = z * (u >= 0.f ? u + 0.5f : sig<EXACT>(u));
}

// Two neighbouring channels.
template <typename T>
struct Pair;
template <>
struct Pair<__nv_bfloat16> {
    typedef __nv_bfloat162 type;
    static __device__ __forceinline__ float2 get(type v) { return __bfloat1622float2(v); }
    static __device__ __forceinline__ type put(float a, float b) { return __floats2bfloat162_rn(a, b); }
};
template <>
struct Pair<float> {
    typedef float2 type;
    static __device__ __forceinline__ float2 get(type v) { return v; }
    static __device__ __forceinline__ type put(float a, float b) { return make_float2(a, b); }
};

// grid (64-channel groups, CTAs of a cluster, portions)
template <typename T>
__global__ void __launch_bounds__(32 * WARPS, 1) gru_scan_kernel(const __grid_constant__ GruArgs a) {
    constexpr bool EXACT = sizeof(T) == 4;
    typedef typename Pair<T>::type T2;
    __shared__ float4 s_part[WARPS][32];           // a warp's stretch: keep and add of both channels
    __shared__ float4 s_cta[2][32];                // this CTA's stretch as a whole, of even and odd turns
    const int rank = blockIdx.y, ctas = gridDim.y;
    cg::cluster_group cl = cg::this_cluster();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, ch = blockIdx.x * 64 + 2 * lane, c = min(ch, a.width - 2);
    pdl_launch();
    pdl_wait();
    const int4 p = a.seg[blockIdx.z];
    float2* st = (float2*)(a.state + (size_t)p.z * a.width + c);
    float2 state = p.w > 0 ? *st : make_float2(0.f, 0.f);      // at the start of this turn's rows; every thread of every CTA keeps it
    const T* x = (const T*)a.x + (size_t)p.x * a.ldx + c;
    T2 rz[STEPS], ru[STEPS], g[STEPS];
    auto fetch = [&](int first) {                  // rows behind the portion repeat its last one
#pragma unroll
        for (int i = 0; i < STEPS; i++) {
            const T* q = x + (size_t)min(first + i, p.y - 1) * a.ldx;
            rz[i] = *(const T2*)q;
            ru[i] = *(const T2*)(q + a.off_u);
            g[i] = *(const T2*)(q + a.off_g);
        }
    };
    auto then = [](float2 s, const float4& v) { return make_float2(fmaf(v.x, s.x, v.z), fmaf(v.y, s.y, v.w)); };
    const int step = STEPS * WARPS * ctas;
    int first = STEPS * (WARPS * rank + warp);
    fetch(first);
    for (int r0 = 0, turn = 0; r0 < p.y; r0 += step, first += step, turn ^= 1) {
        float2 keep[STEPS], add[STEPS], gate[STEPS];
        float4 v = make_float4(1.f, 1.f, 0.f, 0.f);
#pragma unroll
        for (int i = 0; i < STEPS; i++) {
            const float2 z = Pair<T>::get(rz[i]), u = Pair<T>::get(ru[i]), o = Pair<T>::get(g[i]);
            if (EXACT) {
                gates<EXACT>(z.x, u.x, keep[i].x, add[i].x);
                gates<EXACT>(z.y, u.y, keep[i].y, add[i].y);
                gate[i] = make_float2(o.x * sig<EXACT>(o.x), o.y * sig<EXACT>(o.y));
            } else {
                gates3(z.x, u.x, o.x, keep[i].x, add[i].x, gate[i].x);
                gates3(z.y, u.y, o.y, keep[i].y, add[i].y, gate[i].y);
            }
            if (first + i >= p.y) {
                keep[i] = make_float2(1.f, 1.f);
                add[i] = make_float2(0.f, 0.f);
            }
            v.x *= keep[i].x; v.y *= keep[i].y;
            v.z = fmaf(keep[i].x, v.z, add[i].x); v.w = fmaf(keep[i].y, v.w, add[i].y);
        }
        if (r0 + step < p.y) fetch(first + step);  // under way while the stretches are put together
        s_part[warp][lane] = v;
        __syncthreads();
        if (warp == 0) {                           // what comes before every warp's stretch, and the stretch of all
            float4 all = make_float4(1.f, 1.f, 0.f, 0.f);
#pragma unroll 4
            for (int w = 0; w < WARPS; w++) {
                const float4 t = s_part[w][lane];
                s_part[w][lane] = all;
                all = make_float4(all.x * t.x, all.y * t.y, fmaf(t.x, all.z, t.z), fmaf(t.y, all.w, t.w));
            }
            s_cta[turn][lane] = all;
        }
        if (ctas > 1) cl.sync();                   // two sets: nobody writes one before all have passed the turn after its last reading
        else __syncthreads();
        float2 s = state, end = state;             // at this CTA's start; at the end of the turn's rows
        for (int q = 0; q < ctas; q++) {
            if (q == rank) s = end;
            end = then(end, ctas > 1 ? *cl.map_shared_rank(&s_cta[turn][lane], q) : s_cta[turn][lane]);
        }
        s = then(s, s_part[warp][lane]);
        state = end;
        T* o = (T*)a.out + (size_t)(p.x + first) * a.ldo + ch;
#pragma unroll
        for (int i = 0; i < STEPS; i++) {
            s = make_float2(fmaf(keep[i].x, s.x, add[i].x), fmaf(keep[i].y, s.y, add[i].y));
            if (first + i < p.y && ch < a.width) *(T2*)(o + (size_t)i * a.ldo) = Pair<T>::put(s.x * gate[i].x, s.y * gate[i].y);
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
    return a->width < 2 || ((a->width | a->off_u | a->off_g | a->ldx | a->ldo) & 1) || a->off_u < a->width || a->off_g < a->off_u + a->width || a->ldx < a->off_g + a->width || a->ldo < a->width || !a->x || !a->state || !a->out || (((uintptr_t)a->x | (uintptr_t)a->out) & 7);
}

}  // namespace

// Return a cudaError_t value.  max_rows: rows of the longest portion.
B2_API int b2_gru_scan(const GruArgs* a, int n_seg, int max_rows, int f32, int pdl, cudaStream_t st) {
    if (n_seg < 1 || n_seg > 65535 || max_rows < 1 || !a->seg || bad(a)) return (int)cudaErrorInvalidValue;
    GruArgs c = *a;
    void* args[] = {&c};
    int cluster = 1;
    const int groups = (a->width + 63) / 64;       // CTAs for the SMs there are, as far as each has rows
    while (cluster < MAX_CLUSTER && 2 * cluster * groups * n_seg <= 160 && cluster * STEPS * WARPS < max_rows) cluster *= 2;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(groups, cluster, n_seg);
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
