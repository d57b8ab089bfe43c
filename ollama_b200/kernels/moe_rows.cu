// Mixture-of-experts feed-forward of decode steps (one to four rows) over unquantised experts, sm_100a: two launches behind the router's
// product.
//
//   moe_up_rows     picks the experts of a row from its router logits (every CTA for itself), multiplies the row with the gate / up rows of
//                   the chosen experts and of the shared expert, and applies the gated activation
//   moe_down_rows   one product over the concatenated hidden columns of the chosen experts (times their weights) and of the shared one, added
//                   to the residual
//
// A warp owns four consecutive matrix rows; short problems split the row length over KS warps, as in gemv_rows.cu.
#include "choose.cuh"
#include "rows.cuh"

struct MoeUpArgs {
    const float* z;          // [nb][ldz] router logits
    int ldz, n_experts, top; // n_experts: router outputs; scoring: see choose
    const float* h;          // [nb][ldh]
    int ldh, k;              // k: padded row length, a multiple of 8
    const void* w;           // [experts][wrows][k], rows 2i / 2i + 1 = gate / up of hidden column i
    int n, wrows;            // rows used of an expert, rows stored
    const void* ws;          // [ns][k] shared expert, or null
    int ns;
    float limit, limit_s;
    float* out;              // [nb][ldo]: hidden columns of slot s at s * ffp, of the shared expert at top * ffp
    int ldo, ffp;
    int* ids;                // [nb][top]
    float* wts;              // [nb][top]
    const float* correction; // [n_experts] or null
    int real, act;           // router outputs from `real` on stand for the input itself and have no matrices; act: glu_act's number
    ExpertGroups groups;     // count > 0: scores are sigmoids, see choose
};

struct MoeDownArgs {
    const float* a;          // [nb][lda]: as moe_up_rows leaves it; pad columns are zero
    int lda, top, ffp, sfp;  // ffp, sfp: padded hidden sizes, multiples of 8 (sfp 0: no shared expert)
    const int* ids;
    const float* wts;
    const void* w;           // [experts][wrows][ffp]
    const void* ws;          // [.][sfp]
    int n, wrows;            // result columns, rows stored of an expert
    float* x;                // [nb][ldx] (+)= mult * result
    int ldx;
    float mult;
    int store, real;         // store: the result replaces x; real: choices from this one on are the input itself
    const float* h;          // [nb][ldh] that input
    int ldh;
    const float* gate;       // [nb] rows of ldg: the shared expert is multiplied by the sigmoid, or null
    int ldg;
};

namespace {

constexpr int R = 4, MAXJ = 16, MAX_TOP = 16;

// Experts of a row in order of their scores (ties: the lower index) and their weights; by one warp.  Without a correction the scores are the logits and the
// weights the softmax over the chosen ones; with it the softmax over all plus the correction, and that softmax.  With groups the scores are the sigmoids plus the
// correction, inside the groups that are kept, and the weights the chosen sigmoids over their sum, times a factor; `scratch`: 2 n floats of shared memory.
__device__ __forceinline__ void choose(const float* z, const float* correction, int n, int top, int lane, int* ids, float* wts, const ExpertGroups& groups, float* scratch) {
    float v[MAXJ], mz = -INFINITY, total = 0.f;
    const bool sigmoid = groups.count > 0;
    if (sigmoid) {
        for (int e = lane; e < n; e += 32) scratch[e] = sigmoid_exact(z[e]) + (correction ? correction[e] : 0.f);
        __syncwarp();
        keep_groups(scratch, scratch + n, n, groups, lane);
    }
#pragma unroll
    for (int j = 0; j < MAXJ; j++) {
        const int e = lane + 32 * j;
        v[j] = e < n ? (sigmoid ? scratch[e] : z[e]) : -INFINITY;
        mz = fmaxf(mz, v[j]);
    }
    if (correction && !sigmoid) {
        mz = warp_max(mz);
#pragma unroll
        for (int j = 0; j < MAXJ; j++) {
            if (32 * j >= n) break;
            v[j] = expf(v[j] - mz);
            total += v[j];
        }
        total = warp_sum(total);
#pragma unroll
        for (int j = 0; j < MAXJ; j++) {
            if (32 * j >= n) break;
            v[j] = lane + 32 * j < n ? v[j] / total + correction[lane + 32 * j] : -INFINITY;
        }
    }
    float val = -INFINITY;
    int idx = 0;
    for (int s = 0; s < top; s++) {
        float bv = -INFINITY;
        int be = 0x7fffffff;
#pragma unroll
        for (int j = 0; j < MAXJ; j++) {
            if (32 * j >= n) break;
            if (v[j] > bv) {
                bv = v[j];
                be = lane + 32 * j;
            }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
            const int oe = __shfl_xor_sync(0xffffffffu, be, o);
            if (ov > bv || (ov == bv && oe < be)) {
                bv = ov;
                be = oe;
            }
        }
        if (lane == s) {
            val = bv;
            idx = min(be, n - 1);
        }
#pragma unroll
        for (int j = 0; j < MAXJ; j++)
            if (lane + 32 * j == be) v[j] = -INFINITY;
    }
    if (sigmoid) {
        const float w = lane < top ? sigmoid_exact(z[idx]) : 0.f, sum = warp_sum(w) + 1e-20f;
        if (lane < top) {
            ids[lane] = idx;
            wts[lane] = w / sum * groups.scale;
        }
        return;
    }
    if (correction) {
        if (lane < top) {
            ids[lane] = idx;
            wts[lane] = expf(z[idx] - mz) / total;
        }
        return;
    }
    const float mx = __shfl_sync(0xffffffffu, val, 0);
    const float e = lane < top ? expf(val - mx) : 0.f;
    const float sum = warp_sum(e);
    if (lane < top) {
        ids[lane] = idx;
        wts[lane] = e / sum;
    }
}

// 8 consecutive weights times 8 source values
template <bool F32>
struct Piece;
template <>
struct Piece<false> {
    uint4 q;
    __device__ __forceinline__ void load(const void* base, size_t elem) { q = ldg16((const uint8_t*)base + elem * 2); }
    __device__ __forceinline__ float dot(const float (&x)[8]) const {
        const uint32_t w[4] = {q.x, q.y, q.z, q.w};
        float t = 0.f;
#pragma unroll
        for (int i = 0; i < 4; i++) t = fmaf(__uint_as_float(w[i] & 0xffff0000u), x[2 * i + 1], fmaf(__uint_as_float(w[i] << 16), x[2 * i], t));
        return t;
    }
};
template <>
struct Piece<true> {
    uint4 q, q2;
    __device__ __forceinline__ void load(const void* base, size_t elem) {
        q = ldg16((const uint8_t*)base + elem * 4);
        q2 = ldg16((const uint8_t*)base + elem * 4 + 16);
    }
    __device__ __forceinline__ float dot(const float (&x)[8]) const {
        const uint32_t w[8] = {q.x, q.y, q.z, q.w, q2.x, q2.y, q2.z, q2.w};
        float t = 0.f;
#pragma unroll
        for (int i = 0; i < 8; i++) t = fmaf(__uint_as_float(w[i]), x[i], t);
        return t;
    }
};

// grid (row groups / (8 / KS), nb)
template <bool F32, int KS>
__global__ void __launch_bounds__(256) moe_up_rows_kernel(const __grid_constant__ MoeUpArgs a) {
    constexpr int RGS = 8 / KS, U = F32 ? 1 : 2;
    __shared__ int s_id[MAX_TOP];
    __shared__ float s_w[MAX_TOP];
    __shared__ float red[8][R];
    extern __shared__ float scratch[];             // [2 n_experts] with groups
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, rg = warp / KS, ks = warp % KS, b = blockIdx.y;
    pdl_launch();
    pdl_wait();
    if (warp == 0) choose(a.z + (size_t)b * a.ldz, a.correction, a.n_experts, a.top, lane, s_id, s_w, a.groups, scratch);
    __syncthreads();
    if (blockIdx.x == 0 && threadIdx.x < a.top) {
        a.ids[b * a.top + threadIdx.x] = s_id[threadIdx.x];
        a.wts[b * a.top + threadIdx.x] = s_w[threadIdx.x];
    }
    const int per = (a.n + R - 1) / R, sgroups = (a.ns + R - 1) / R;
    int g = blockIdx.x * RGS + rg;
    const bool active = g < per * a.top + sgroups;
    const bool shared = g >= per * a.top;
    const int slot = active && !shared ? g / per : a.top;
    g -= slot * per;
    const int n = shared ? a.ns : a.n, row0 = active ? g * R : 0;
    const void* base = shared || !active ? a.ws : a.w;
    const size_t first = shared || !active ? 0 : (size_t)s_id[slot] * a.wrows;
    float acc[R] = {};
    if (active && (shared || s_id[slot] < a.real)) {
        const float* x = a.h + (size_t)b * a.ldh;
        const int pieces = a.k >> 3, step = KS * 32;
        for (int p0 = ks * 32 + lane; p0 < pieces; p0 += U * step) {
            Piece<F32> w[U][R];
#pragma unroll
            for (int u = 0; u < U; u++)
                if (p0 + u * step < pieces) {
#pragma unroll
                    for (int r = 0; r < R; r++) w[u][r].load(base, (first + min(row0 + r, n - 1)) * a.k + (size_t)(p0 + u * step) * 8);
                }
#pragma unroll
            for (int u = 0; u < U; u++) {
                const int p = p0 + u * step;
                if (p >= pieces) continue;
                float xv[8];
                *(float4*)xv = *(const float4*)(x + 8 * p);
                *(float4*)(xv + 4) = *(const float4*)(x + 8 * p + 4);
#pragma unroll
                for (int r = 0; r < R; r++) acc[r] += w[u][r].dot(xv);
            }
        }
    }
#pragma unroll
    for (int r = 0; r < R; r++) {
        acc[r] = warp_sum(acc[r]);
        if (lane == 0) red[warp][r] = acc[r];
    }
    __syncthreads();
    if (ks == 0 && active && lane < R / 2 && row0 + 2 * lane < n) {
        float v0 = 0.f, v1 = 0.f;
#pragma unroll
        for (int j = 0; j < KS; j++) {
            v0 += red[rg * KS + j][2 * lane];
            v1 += red[rg * KS + j][2 * lane + 1];
        }
        const float limit = shared ? a.limit_s : a.limit;
        const float y = F32 ? glu_act_exact(v0, v1, a.act, SWIGLU_ALPHA, limit) : glu_act(v0, v1, a.act, SWIGLU_ALPHA, limit);
        a.out[(size_t)b * a.ldo + (size_t)slot * a.ffp + (row0 >> 1) + lane] = y;
    }
}

template <bool F32, int KS>
__global__ void __launch_bounds__(256) moe_down_rows_kernel(const __grid_constant__ MoeDownArgs a) {
    constexpr int RGS = 8 / KS, U = F32 ? 1 : 2;
    __shared__ int s_id[MAX_TOP];
    __shared__ float s_w[MAX_TOP];
    __shared__ float red[8][R];
    float same = 0.f;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, rg = warp / KS, ks = warp % KS, b = blockIdx.y;
    const int row0 = (blockIdx.x * RGS + rg) * R;
    const bool active = row0 < a.n;
    pdl_launch();
    pdl_wait();
    if (threadIdx.x < a.top) {
        s_id[threadIdx.x] = a.ids[b * a.top + threadIdx.x];
        s_w[threadIdx.x] = a.wts[b * a.top + threadIdx.x];
    }
    __syncthreads();
    float acc[R] = {};
    if (active) {
        const float* x = a.a + (size_t)b * a.lda;
        const float sw = a.gate && a.sfp ? (F32 ? sigmoid_exact(a.gate[(size_t)b * a.ldg]) : sigmoid_f(a.gate[(size_t)b * a.ldg])) : 1.f;
        for (int s = 0; s < a.top; s++)
            if (s_id[s] >= a.real) same += s_w[s];
        const int f8 = a.ffp >> 3, routed = a.top * f8, pieces = routed + (a.sfp >> 3), step = KS * 32;
        for (int p0 = ks * 32 + lane; p0 < pieces; p0 += U * step) {
            Piece<F32> w[U][R];
            float f[U];
#pragma unroll
            for (int u = 0; u < U; u++) {
                const int p = p0 + u * step;
                f[u] = 0.f;
                if (p >= pieces || (p < routed && s_id[p / f8] >= a.real)) continue;
                const bool shared = p >= routed;
                const int slot = shared ? 0 : p / f8, c = 8 * (shared ? p - routed : p - slot * f8), ld = shared ? a.sfp : a.ffp;
                const void* base = shared ? a.ws : a.w;
                const size_t first = shared ? 0 : (size_t)s_id[slot] * a.wrows;
                f[u] = shared ? sw : s_w[slot];
#pragma unroll
                for (int r = 0; r < R; r++) w[u][r].load(base, (first + min(row0 + r, a.n - 1)) * ld + c);
            }
#pragma unroll
            for (int u = 0; u < U; u++) {
                const int p = p0 + u * step;
                if (p >= pieces || f[u] == 0.f) continue;
                float xv[8];
                *(float4*)xv = *(const float4*)(x + 8 * p);
                *(float4*)(xv + 4) = *(const float4*)(x + 8 * p + 4);
#pragma unroll
                for (int r = 0; r < R; r++) acc[r] = fmaf(f[u], w[u][r].dot(xv), acc[r]);
            }
        }
    }
#pragma unroll
    for (int r = 0; r < R; r++) {
        acc[r] = warp_sum(acc[r]);
        if (lane == 0) red[warp][r] = acc[r];
    }
    __syncthreads();
    if (ks == 0 && active && lane < R && row0 + lane < a.n) {
        float v = 0.f;
#pragma unroll
        for (int j = 0; j < KS; j++) v += red[rg * KS + j][lane];
        if (same != 0.f) v = fmaf(same, a.h[(size_t)b * a.ldh + row0 + lane], v);
        float* o = a.x + (size_t)b * a.ldx + row0 + lane;
        *o = a.store ? a.mult * v : *o + a.mult * v;
    }
}

// Warps that share a row group: until `want` warps carry loads, as far as a lane keeps two pieces.
int split_of(long groups, int pieces, long want) {
    int ks = 1;
    while (ks < 8 && groups * ks < want && pieces / (64 * ks) >= 1) ks <<= 1;
    return ks;
}

#define B2_PICK_KS(fn, f32, ks)                                                                                      \
    (f32 ? (ks == 8 ? (const void*)fn<true, 8> : ks == 4 ? (const void*)fn<true, 4> : ks == 2 ? (const void*)fn<true, 2> : (const void*)fn<true, 1>) \
         : (ks == 8 ? (const void*)fn<false, 8> : ks == 4 ? (const void*)fn<false, 4> : ks == 2 ? (const void*)fn<false, 2> : (const void*)fn<false, 1>))

}  // namespace

// Return a cudaError_t value.
B2_API int b2_moe_up_rows(const MoeUpArgs* a, int nb, int f32, int pdl, cudaStream_t st) {
    if (nb < 1 || nb > 65535 || a->n_experts < 1 || a->n_experts > 32 * MAXJ || a->top < 1 || a->top > MAX_TOP || a->top > a->n_experts || a->k < 8 || (a->k & 7) || (a->ldh & 3) ||
        a->n < 2 || (a->n & 1) || a->wrows < a->n || (a->ns & 1) || (a->ns && !a->ws) || a->ffp < a->n / 2 || a->ldo < a->top * a->ffp + a->ns / 2 || ((uintptr_t)a->h & 15) ||
        ((uintptr_t)a->w & 15) || ((uintptr_t)a->ws & 15) || a->real < 1 || a->real > a->n_experts || a->act < 0 || a->act > 2 || a->groups.count < 0 ||
        (a->groups.count && (a->n_experts % a->groups.count || a->groups.keep < 1 || a->top > a->n_experts / a->groups.count * a->groups.keep)))
        return (int)cudaErrorInvalidValue;
    const long groups = (long)a->top * ((a->n + R - 1) / R) + (a->ns + R - 1) / R;
    const int ks = split_of(groups * nb, a->k >> 3, 1800), rgs = 8 / ks;
    MoeUpArgs c = *a;
    void* args[] = {&c};
    return launch_rows(B2_PICK_KS(moe_up_rows_kernel, f32, ks), dim3((unsigned)((groups + rgs - 1) / rgs), nb), dim3(256), a->groups.count ? (size_t)a->n_experts * 8 : 0, args, st,
                       pdl);
}

B2_API int b2_moe_down_rows(const MoeDownArgs* a, int nb, int f32, int pdl, cudaStream_t st) {
    if (nb < 1 || nb > 65535 || a->top < 1 || a->top > MAX_TOP || a->ffp < 8 || (a->ffp & 7) || (a->sfp & 7) || (a->sfp && !a->ws) || a->n < 1 || a->wrows < a->n || (a->lda & 3) ||
        a->lda < a->top * a->ffp + a->sfp || ((uintptr_t)a->a & 15) || ((uintptr_t)a->w & 15) || ((uintptr_t)a->ws & 15) || a->real < 1)
        return (int)cudaErrorInvalidValue;
    const long groups = (a->n + R - 1) / R;
    const int ks = split_of(groups * nb, (a->top * a->ffp + a->sfp) >> 3, 16000), rgs = 8 / ks;
    MoeDownArgs c = *a;
    void* args[] = {&c};
    return launch_rows(B2_PICK_KS(moe_down_rows_kernel, f32, ks), dim3((unsigned)((groups + rgs - 1) / rgs), nb), dim3(256), 0, args, st, pdl);
}
