// Matrix-vector products of decode steps over unquantised weights (bf16, or fp32 for 32-bit models), 1..4 rows, with what
// surrounds them in a layer fused in, sm_100a.
//
// Up to four matrices share one launch and one source row.  The source is read in one of four ways:
//   rows     fp32 activations as they are;
//   norm     RMS-normalised: every segment has a norm weight of its own (branches of a parallel block), the weight is multiplied
//            into the row while the dot products run and the row's 1 / rms, which every CTA computes, into the results;
//   layer    layer-normalised: the same, and the results less mean times the matrix row's weighted sum, plus the row's product with the
//            bias, both made at load;
//   joined   two rows side by side;
// The epilogue applies an activation (of single rows, or of gate / up pairs), a factor, and stores or accumulates (the residual add).  The first rows of one matrix may also run
// through a causal depthwise convolution, with or without SiLU, with the slot's last inputs, which are shifted here or by the kernel that advances the
// recurrence.  A warp owns four consecutive rows of a matrix and strides over their 16-byte pieces; short problems split the row
// length over KS warps of the CTA.  Weight rows are requested from L2 before the grid-dependency wait (they do not depend on the producer
// kernel).  One group of rows per warp measured faster than resident CTAs that walk over groups (5.5 against 4.7 TB/s on 184 MB).
#include "rows.cuh"

struct RowSeg {
    const void* w;       // [n][ldw]
    const float* g;      // [k] norm weight (norm source)
    const float* rs;     // [n] sum of w g over the row (layer norm)
    const float* rc;     // [n] added to the result, or null
    float* out;          // [nb][ldo]
    int n, ldw, ldo;
    int act;             // out_act's number, or GLU_BASE + glu_act's: rows 2i / 2i + 1 are gate / up of output i
    int accumulate;
    float alpha, limit;  // factor of the result; limit of the clamped gated unit
    const void* mul;     // result times mul[mul_row[b] * ldm + row] in the weights' type, after the activation; or null
    int ldm;
    float act_p, act_q;  // numbers of the activation, where it has some
};

enum RowSrc : int { SRC_ROWS = 0, SRC_NORM = 1, SRC_JOINED = 2, SRC_LAYER = 3 };

__host__ __device__ constexpr bool norm_source(int src) { return src == SRC_NORM || src == SRC_LAYER; }

struct GemvRowsArgs {
    RowSeg seg[4];
    int nseg, nb, k;     // k: padded row length, a multiple of 8 (source columns beyond the true length are zero)
    int src, f32;        // source kind, weight type (0 bf16, 1 fp32)
    const float* x;      // [nb][ldx]
    int ldx;
    const float* x2;     // joined: columns k1 .. k - 1
    int ldx2, k1;
    float eps;
    int kn;              // norm: true row length
    // convolution of the rows 0 .. conv_n - 1 of matrix conv_seg (conv_seg < 0: none)
    int conv_seg, conv_n, taps;
    const float* conv_w;          // [taps][conv_n], last tap = current token
    const float* conv_b;          // [conv_n] or null
    float* conv_state;            // [slots][taps - 1][conv_n], oldest first
    int conv_silu, conv_shift;    // conv_shift: the state is moved on here
    float* conv_out;              // [nb][ldu]
    int ldu;
    const int* slots;
    const int* positions;         // 0: the state counts as zeros
    // norm sources: the normalised row of matrix 0 as a result of its own (h = null: none)
    float* h;                     // [nb][ldh], k columns
    int ldh;
    const float* hb;              // [k] layer norm's bias
    const int* mul_row;           // [nb]
};

namespace {

constexpr int R = 4;

template <int NB, int SRC>
__device__ __forceinline__ void source8(const GemvRowsArgs& a, const float* g, int col, float (&x)[NB][8]) {
    float gv[8];
    if (norm_source(SRC)) {
        *(float4*)gv = __ldg((const float4*)(g + col));
        *(float4*)(gv + 4) = __ldg((const float4*)(g + col + 4));
    }
#pragma unroll
    for (int b = 0; b < NB; b++) {
        const int bb = b < a.nb ? b : 0;
        const float* p = a.x + (size_t)bb * a.ldx + col;
        if (SRC == SRC_JOINED && col >= a.k1) p = a.x2 + (size_t)bb * a.ldx2 + col - a.k1;
        *(float4*)x[b] = *(const float4*)p;
        *(float4*)(x[b] + 4) = *(const float4*)(p + 4);
        if (norm_source(SRC)) {
#pragma unroll
            for (int i = 0; i < 8; i++) x[b][i] *= gv[i];
        }
    }
}

template <int NB, int SRC, bool F32, int KS>
__global__ void __launch_bounds__(256, NB == 1 ? 3 : NB == 2 ? 4 : 2) gemv_rows_kernel(const __grid_constant__ GemvRowsArgs a) {
    constexpr int RGS = 8 / KS;
    constexpr int EB = F32 ? 4 : 2;
    constexpr int U = F32 || NB == 2 ? 1 : 2;           // pieces in flight per row
    __shared__ float red[8][R * NB];
    __shared__ float s_ss[8][NB], s_sm[8][NB];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int rg = warp / KS, ks = warp % KS;
    const uint8_t* wp[R];
    int g = blockIdx.x * RGS + rg, s = 0;
    for (; s < a.nseg; s++) {
        const int groups = (a.seg[s].n + R - 1) / R;
        if (g < groups) break;
        g -= groups;
    }
    const bool active = s < a.nseg;
    const RowSeg& w = a.seg[active ? s : 0];
    const int row0 = active ? g * R : 0;
#pragma unroll
    for (int r = 0; r < R; r++) wp[r] = (const uint8_t*)w.w + (size_t)min(row0 + r, w.n - 1) * w.ldw * EB;
    pdl_launch();
    if (active) {
        for (int off = (ks * 32 + lane) * 128; off < a.k * EB; off += KS * 32 * 128) {
#pragma unroll
            for (int r = 0; r < R; r++) asm volatile("prefetch.global.L2 [%0];" ::"l"(wp[r] + off));
        }
    }
    pdl_wait();
    if (norm_source(SRC)) {
#pragma unroll
        for (int b = 0; b < NB; b++) {
            const float* x = a.x + (size_t)(b < a.nb ? b : 0) * a.ldx;
            float ss = 0.f, sm = 0.f;
            for (int i = 4 * threadIdx.x; i < a.k; i += 1024) {      // columns beyond the true length are zero
                const float4 v = *(const float4*)(x + i);
                ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
                if (SRC == SRC_LAYER) sm += v.x + v.y + v.z + v.w;
            }
            ss = warp_sum(ss);
            if (SRC == SRC_LAYER) sm = warp_sum(sm);
            if (lane == 0) {
                s_ss[warp][b] = ss;
                if (SRC == SRC_LAYER) s_sm[warp][b] = sm;
            }
        }
    }
    float acc[R][NB];
#pragma unroll
    for (int r = 0; r < R; r++)
#pragma unroll
        for (int b = 0; b < NB; b++) acc[r][b] = 0.f;
    if (active) {
        const int pieces = a.k >> 3, step = KS * 32;
        for (int p0 = ks * 32 + lane; p0 < pieces; p0 += U * step) {
            uint4 wv[U][R], wv2[U][R];
#pragma unroll
            for (int u = 0; u < U; u++) {
                const int p = p0 + u * step;
                if (p < pieces) {
#pragma unroll
                    for (int r = 0; r < R; r++) {
                        wv[u][r] = ldg16(wp[r] + (size_t)p * 8 * EB);
                        if (F32) wv2[u][r] = ldg16(wp[r] + (size_t)p * 8 * EB + 16);
                    }
                }
            }
#pragma unroll
            for (int u = 0; u < U; u++) {
                const int p = p0 + u * step;
                if (p >= pieces) continue;
                float x[NB][8];
                source8<NB, SRC>(a, w.g, 8 * p, x);
#pragma unroll
                for (int r = 0; r < R; r++) {
                    float wf[8];
                    const uint32_t q[4] = {wv[u][r].x, wv[u][r].y, wv[u][r].z, wv[u][r].w};
                    if (F32) {
                        const uint32_t q2[4] = {wv2[u][r].x, wv2[u][r].y, wv2[u][r].z, wv2[u][r].w};
#pragma unroll
                        for (int i = 0; i < 4; i++) {
                            wf[i] = __uint_as_float(q[i]);
                            wf[4 + i] = __uint_as_float(q2[i]);
                        }
                    } else {
#pragma unroll
                        for (int i = 0; i < 4; i++) {
                            wf[2 * i] = __uint_as_float(q[i] << 16);
                            wf[2 * i + 1] = __uint_as_float(q[i] & 0xffff0000u);
                        }
                    }
#pragma unroll
                    for (int b = 0; b < NB; b++) {
                        float t = 0.f;
#pragma unroll
                        for (int i = 0; i < 8; i++) t = fmaf(wf[i], x[b][i], t);
                        acc[r][b] += t;
                    }
                }
            }
        }
    }
#pragma unroll
    for (int r = 0; r < R; r++)
#pragma unroll
        for (int b = 0; b < NB; b++) {
            acc[r][b] = warp_sum(acc[r][b]);
            if (lane == 0) red[warp][r * NB + b] = acc[r][b];
        }
    __syncthreads();
    auto row_stats = [&](int b, float& mean, float& inv) {
        float ss = 0.f, sm = 0.f;
#pragma unroll
        for (int i = 0; i < 8; i++) {
            ss += s_ss[i][b];
            if (SRC == SRC_LAYER) sm += s_sm[i][b];
        }
        mean = SRC == SRC_LAYER ? sm / (float)a.kn : 0.f;
        inv = 1.f / sqrtf((SRC == SRC_LAYER ? fmaxf(ss / (float)a.kn - mean * mean, 0.f) : ss / (float)a.kn) + a.eps);
    };
    if (norm_source(SRC) && a.h) {          // a slice of the normalised rows per CTA
        for (int i = blockIdx.x * 256 + threadIdx.x; i < a.nb * a.k; i += gridDim.x * 256) {
            const int b = i / a.k, c = i - b * a.k;
            float mean, inv;
            row_stats(b, mean, inv);
            a.h[(size_t)b * a.ldh + c] = (a.x[(size_t)b * a.ldx + c] - mean) * inv * a.seg[0].g[c] + (a.hb ? a.hb[c] : 0.f);
        }
    }
    const int r = lane / NB, b = lane % NB, row = row0 + r;
    if (ks != 0 || !active) return;
    const bool mine = lane < R * NB && row < w.n && b < a.nb;
    float v = 0.f;
    if (mine) {
#pragma unroll
        for (int k2 = 0; k2 < KS; k2++) v += red[rg * KS + k2][lane];
        if (norm_source(SRC)) {
            float mean, inv;
            row_stats(b, mean, inv);
            v = SRC == SRC_LAYER ? (v - mean * w.rs[row]) * inv : v * inv;
        }
        if (w.rc) v += w.rc[row];
    }
    if (w.act >= GLU_BASE) {
        const float up = __shfl_down_sync(0xffffffffu, v, NB);
        if (mine && !(r & 1)) {
            const float y = F32 ? glu_act_exact(v, up, w.act - GLU_BASE, SWIGLU_ALPHA, w.limit) : glu_act(v, up, w.act - GLU_BASE, SWIGLU_ALPHA, w.limit);
            w.out[(size_t)b * w.ldo + (row >> 1)] = y;
        }
        return;
    }
    if (mine) {
        v = out_act<F32>(v, w.act, w.act_p, w.act_q);
        if (w.mul) {
            const size_t m = (size_t)a.mul_row[b] * w.ldm + row;
            v *= F32 ? ((const float*)w.mul)[m] : __bfloat162float(((const __nv_bfloat16*)w.mul)[m]);
        }
        float* o = w.out + (size_t)b * w.ldo + row;
        *o = w.accumulate ? *o + w.alpha * v : w.alpha * v;
        if (s == a.conv_seg && row < a.conv_n) {
            float u = (a.conv_b ? a.conv_b[row] : 0.f) + a.conv_w[(size_t)(a.taps - 1) * a.conv_n + row] * v;
            const bool old = a.positions[b] > 0;
            float* st = a.conv_state + (size_t)a.slots[b] * (a.taps - 1) * a.conv_n + row;
            for (int j = 0; j < a.taps - 1; j++) {
                const float in = old ? st[(size_t)j * a.conv_n] : 0.f;
                u += in * a.conv_w[(size_t)j * a.conv_n + row];
                if (a.conv_shift && j > 0) st[(size_t)(j - 1) * a.conv_n] = in;
            }
            if (a.conv_shift && a.taps > 1) st[(size_t)(a.taps - 2) * a.conv_n] = v;
            a.conv_out[(size_t)b * a.ldu + row] = a.conv_silu ? silu_f(u) : u;
        }
    }
}

template <int NB, int SRC, bool F32>
const void* pick_ks(int ks) {
    switch (ks) {
        case 8: return (const void*)gemv_rows_kernel<NB, SRC, F32, 8>;
        case 4: return (const void*)gemv_rows_kernel<NB, SRC, F32, 4>;
        case 2: return (const void*)gemv_rows_kernel<NB, SRC, F32, 2>;
        default: return (const void*)gemv_rows_kernel<NB, SRC, F32, 1>;
    }
}
template <int SRC, bool F32>
const void* pick_nb(int nb, int ks) {
    return nb <= 1 ? pick_ks<1, SRC, F32>(ks) : nb <= 2 ? pick_ks<2, SRC, F32>(ks) : pick_ks<4, SRC, F32>(ks);
}
template <bool F32>
const void* pick_src(int src, int nb, int ks) {
    switch (src) {
        case SRC_NORM: return pick_nb<SRC_NORM, F32>(nb, ks);
        case SRC_LAYER: return pick_nb<SRC_LAYER, F32>(nb, ks);
        case SRC_JOINED: return pick_nb<SRC_JOINED, F32>(nb, ks);
        default: return pick_nb<SRC_ROWS, F32>(nb, ks);
    }
}

}  // namespace

// Returns a cudaError_t value.
B2_API int b2_gemv_rows(const GemvRowsArgs* a, int pdl, cudaStream_t st) {
    if (a->nb < 1 || a->nb > 4 || a->nseg < 1 || a->nseg > 4 || a->k < 8 || (a->k & 7) || !a->x || (a->ldx & 3) || ((uintptr_t)a->x & 15) || a->src < 0 || a->src > SRC_LAYER)
        return (int)cudaErrorInvalidValue;
    if (a->src == SRC_JOINED && (!a->x2 || (a->ldx2 & 3) || ((uintptr_t)a->x2 & 15) || (a->k1 & 7))) return (int)cudaErrorInvalidValue;
    if (a->conv_seg >= 0 && (a->conv_seg >= a->nseg || a->conv_n < 1 || a->conv_n > a->seg[a->conv_seg].n || a->taps < 1 || !a->conv_w || !a->conv_state ||
                             !a->conv_out || !a->slots || !a->positions))
        return (int)cudaErrorInvalidValue;
    if (a->h && !norm_source(a->src)) return (int)cudaErrorInvalidValue;
    long groups = 0;
    for (int s = 0; s < a->nseg; s++) {
        const RowSeg& w = a->seg[s];
        if (!w.w || !w.out || w.n < 1 || w.ldw < a->k || (w.ldw & 7) || ((uintptr_t)w.w & 15) || (norm_source(a->src) && (!w.g || ((uintptr_t)w.g & 15) || (a->src == SRC_LAYER && !w.rs))) ||
            w.act < 0 || (w.act > ACT_LAST && w.act < GLU_BASE) || w.act > GLU_BASE + 2 || (w.act >= GLU_BASE && ((w.n & 1) || w.mul)) || (w.mul && !a->mul_row))
            return (int)cudaErrorInvalidValue;
        groups += (w.n + R - 1) / R;
    }
    // Split the row length over KS warps until there are warps enough for the loads in flight, as far as a lane keeps two pieces; and long
    // rows further, down to four to eight pieces a lane (sweep over 2048 .. 11008 columns and 2048 .. 32768 rows).
    const int pieces = a->k >> 3, enough = a->nb <= 2 && pieces >= 512 ? 4 : 8;
    const long want = a->nb == 2 ? 3600 : 1800;
    int ks = 1;
    while (ks < 8 && ((groups * ks < want && pieces / (64 * ks) >= 1) || pieces / (64 * ks) >= enough)) ks <<= 1;
    const int rgs = 8 / ks;
    GemvRowsArgs copy = *a;
    void* args[] = {&copy};
    const void* fn = a->f32 ? pick_src<true>(a->src, a->nb, ks) : pick_src<false>(a->src, a->nb, ks);
    return launch_rows(fn, dim3((unsigned)((groups + rgs - 1) / rgs)), dim3(256), 0, args, st, pdl);
}
