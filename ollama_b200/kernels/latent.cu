// Latent attention on a paged cache, sm_100a: everything around the scores.
//
// A position's cache row is [latent, padded to CP | rotated key part shared by all heads | zeros up to W]; pages of 64 rows as in
// attn_paged.cu with one key head.  Per head the key is [U_h c | rotated part] and the value V_h c, so a query row may be taken into the
// latent space instead, q . (U_h c) = (U_h^T q) . c, and the weighted sum of latents out of it, V_h (sum p c): attention then reads each
// cache row once for all heads ("absorbed" form: decode steps, short portions, 32-bit models).  Long prompt portions multiply U and V
// out for the visible positions instead, which costs fewer products per score.
//
//   latent_step    a row's latent under its RMS norm and rotated key part into the cache; U_h^T q and the rotated query part
//   latent_merge   the split results of the absorbed form added up and multiplied by V_h (a few rows); latent_reduce and latent_values: the
//                  same in two launches, the second on the tensor cores with 16 rows at a time
//   latent_gather  cache rows of whole sequences side by side, for the products of the long form
//   latent_rows    cache rows and query rows of the long form
//
// Rows: `rows` lists the rows of a step that a launch is for (null: all); results are stored in the order of that list, except
// where noted.
#include "rows.cuh"

struct LatentStepArgs {
    const float* q;          // [.][ldq]: per head dim unrotated | rot rotated values
    const float* c;          // [.][ldc]: the latent, then the rotated key part
    int ldq, ldc, n_heads, dim, rot, rank;
    const float* norm;       // [rank] weight of the latent's norm
    float eps;
    const double* freqs;     // [rot / 2]
    int interleaved;         // rotary pairs (2i, 2i + 1) instead of (i, i + rot / 2)
    const int* rows;
    const int* positions;    // of the step's rows
    const int* slots;
    const int* page_table;   // [slots][max_pages]
    int max_pages;
    void* cache;             // [pages][64][w]
    int cp, w, cache32;      // padded latent, row length; element type f16 or fp32
    int append;              // write the cache rows
    const void* uk;          // [heads][dim][cp], bf16 or (w32) fp32; null: no queries
    int w32;
    void* q_out;             // [n][heads][w] in the cache's type; long form: [n][heads][dp + rp] f16, unrotated part, zeros, rotated part, zeros
    int dp, rp;              // long form (uk null)
    float mscale;            // factor of cosines and sines
};

struct LatentMergeArgs {
    const float* acc;        // [n][heads][splits][cp]
    const float2* ml;        // [n][heads][splits] (max, sum; a sum of 0: nothing there), or null: one split, normalised
    int n_heads, splits, cp, vdim;
    const void* uv;          // [heads * vdim][cp]
    int w32;
    const int* rows;         // the result of list entry i goes to row rows[i]
    void* out;               // [.][ldo], head h at column h * vdim
    int ldo, out16;
};

struct LatentGatherArgs {
    const __half* cache;
    int cp, w, rot;
    const int4* seqs;        // (result row of position 0, end of the positions, slot, first position)
    const int* page_table;
    int max_pages;
    __nv_bfloat16* c;        // [.][cp]
    __half* r;               // [.][rp] rotated key part, zero-padded
    int rp;
};

namespace {

// One CTA: cache row of step row r and, with q set, the rotated parts of its queries (rows of w values, cp behind their start) and the zeros
// behind them.  `cs` holds rot floats.
template <typename CT>
__device__ __forceinline__ void append_row(const LatentStepArgs& a, int r, CT* q, float* cs, float* red) {
    const int tid = threadIdx.x, nt = blockDim.x, pos = a.positions[r], slot = a.slots[r], half = a.rot >> 1, pad = a.w - a.cp;
    const float* row = a.q + (size_t)r * a.ldq;
    const float* c = a.c + (size_t)r * a.ldc;
    float ss = 0.f;
#pragma unroll 4
    for (int i = tid; i < a.rank; i += nt) ss += c[i] * c[i];
    ss = warp_sum(ss);
    if ((tid & 31) == 0) red[tid >> 5] = ss;
    for (int i = tid; i < half; i += nt) {
        float sn, co;
        sincosf(rot_angle(pos, a.freqs[i]), &sn, &co);
        cs[i] = co * a.mscale;
        cs[half + i] = sn * a.mscale;
    }
    __syncthreads();
    ss = 0.f;
    for (int i = 0; i < nt >> 5; i++) ss += red[i];
    const float inv = 1.f / sqrtf(ss / (float)a.rank + a.eps);
    auto rotated = [&](const float* v, int i) {
        const bool first = a.interleaved ? !(i & 1) : i < half;
        const int p = a.interleaved ? i >> 1 : (first ? i : i - half);
        const float other = v[a.interleaved ? i ^ 1 : (first ? i + half : i - half)];
        return first ? v[i] * cs[p] - other * cs[half + p] : v[i] * cs[p] + other * cs[half + p];
    };
    if (a.append) {
        CT* o = (CT*)a.cache + paged_row(a.page_table + (size_t)slot * a.max_pages, pos, 1, 0) * a.w;
#pragma unroll 4
        for (int i = tid; i < a.cp; i += nt) o[i] = from_f<CT>(i < a.rank ? c[i] * inv * a.norm[i] : 0.f);
        for (int i = tid; i < pad; i += nt) o[a.cp + i] = from_f<CT>(i < a.rot ? rotated(c + a.rank, i) : 0.f);
    }
    if (q) {
#pragma unroll 4
        for (int j = tid; j < a.n_heads * pad; j += nt) {
            const int h = j / pad, i = j - h * pad;
            q[(size_t)h * a.w + a.cp + i] = from_f<CT>(i < a.rot ? rotated(row + (size_t)h * (a.dim + a.rot) + a.dim, i) : 0.f);
        }
    }
}

template <typename WT>
__device__ __forceinline__ void load8(const WT* p, float (&f)[8]);
template <>
__device__ __forceinline__ void load8<float>(const float* p, float (&f)[8]) {
    *(float4*)f = __ldg((const float4*)p);
    *(float4*)(f + 4) = __ldg((const float4*)p + 1);
}
template <>
__device__ __forceinline__ void load8<__nv_bfloat16>(const __nv_bfloat16* p, float (&f)[8]) {
    const uint4 v = __ldg((const uint4*)p);
    const uint32_t q[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; i++) {
        f[2 * i] = __uint_as_float(q[i] << 16);
        f[2 * i + 1] = __uint_as_float(q[i] & 0xffff0000u);
    }
}

constexpr int COLS = 128;      // latent columns of a CTA of latent_step
constexpr int DG = 16;         // groups of d values, one partial sum each

// grid (heads * column parts + NB, row groups of NB): the last NB CTAs of a row group do what belongs to a row, the others form U^T q
template <typename CT, typename WT, int NB>
__global__ void __launch_bounds__(256) latent_step_kernel(const __grid_constant__ LatentStepArgs a, int n) {
    extern __shared__ float sq[];                  // [NB][dim], or the rotation's cosines and sines
    __shared__ float red[DG][COLS + 4];
    const int tid = threadIdx.x, i0 = blockIdx.y * NB;
    const int parts = (a.cp + COLS - 1) / COLS;
    const int h = blockIdx.x / parts, part = blockIdx.x % parts;
    const int rb = (int)blockIdx.x - a.n_heads * parts;            // >= 0: row of the group
    const int cg = tid & 15, dg = tid >> 4, col = part * COLS + 8 * cg;
    const WT* u = (const WT*)a.uk + ((size_t)h * a.dim) * a.cp + col;
    pdl_launch();
    if (rb < 0 && col < a.cp && (cg & 7) == 0)
        for (int d = dg; d < a.dim; d += DG) asm volatile("prefetch.global.L2 [%0];" ::"l"(u + (size_t)d * a.cp));
    pdl_wait();
    if (rb >= 0) {
        if (i0 + rb < n) append_row<CT>(a, a.rows ? a.rows[i0 + rb] : i0 + rb, (CT*)a.q_out + (size_t)(i0 + rb) * a.n_heads * a.w, sq, &red[0][0]);
        return;
    }
    const int nb = min(NB, n - i0), dq = a.dim + a.rot;
    for (int j = tid; j < nb * a.dim; j += 256) {
        const int b = j / a.dim, d = j - b * a.dim, r = a.rows ? a.rows[i0 + b] : i0 + b;
        sq[b * a.dim + d] = a.q[(size_t)r * a.ldq + (size_t)h * dq + d];
    }
    __syncthreads();
    float acc[NB][8];
#pragma unroll
    for (int b = 0; b < NB; b++)
#pragma unroll
        for (int e = 0; e < 8; e++) acc[b][e] = 0.f;
    if (col < a.cp) {
#pragma unroll 4
        for (int d = dg; d < a.dim; d += DG) {
            float w[8];
            load8<WT>(u + (size_t)d * a.cp, w);
#pragma unroll
            for (int b = 0; b < NB; b++) {
                const float q = b < nb ? sq[b * a.dim + d] : 0.f;
#pragma unroll
                for (int e = 0; e < 8; e++) acc[b][e] = fmaf(q, w[e], acc[b][e]);
            }
        }
    }
#pragma unroll
    for (int b = 0; b < NB; b++) {
        if (b >= nb) break;
        __syncthreads();
        *(float4*)&red[dg][8 * cg] = make_float4(acc[b][0], acc[b][1], acc[b][2], acc[b][3]);
        *(float4*)&red[dg][8 * cg + 4] = make_float4(acc[b][4], acc[b][5], acc[b][6], acc[b][7]);
        __syncthreads();
        const int c = part * COLS + tid;
        if (tid < COLS && c < a.cp) {
            float s = 0.f;
#pragma unroll
            for (int g = 0; g < DG; g++) s += red[g][tid];
            ((CT*)a.q_out)[((size_t)(i0 + b) * a.n_heads + h) * a.w + c] = from_f<CT>(s);
        }
    }
}

// One CTA per row.
__global__ void __launch_bounds__(256) latent_rows_kernel(const __grid_constant__ LatentStepArgs a) {
    extern __shared__ float cs[];
    __shared__ float red[8];
    const int i = blockIdx.x, r = a.rows ? a.rows[i] : i, half = a.rot >> 1, dk = a.dp + a.rp, dk2 = dk >> 1;
    pdl_launch();
    pdl_wait();
    append_row<__half>(a, r, nullptr, cs, red);
    const float* q = a.q + (size_t)r * a.ldq;
    __half* o = (__half*)a.q_out + (size_t)i * a.n_heads * dk;
    for (int j = threadIdx.x; j < a.n_heads * dk2; j += 256) {      // two neighbouring values
        const int h = j / dk2, c = 2 * (j - h * dk2);
        const float* qh = q + (size_t)h * (a.dim + a.rot);
        float v[2];
#pragma unroll
        for (int e = 0; e < 2; e++) {
            const int d = c + e - a.dp;
            if (c + e < a.dim) v[e] = qh[c + e];
            else if (d < 0 || d >= a.rot) v[e] = 0.f;
            else {
                const float* t = qh + a.dim;
                const bool first = a.interleaved ? !(d & 1) : d < half;
                const int p = a.interleaved ? d >> 1 : (first ? d : d - half);
                const float y = t[a.interleaved ? d ^ 1 : (first ? d + half : d - half)];
                v[e] = first ? t[d] * cs[p] - y * cs[half + p] : t[d] * cs[p] + y * cs[half + p];
            }
        }
        *(__half2*)(o + (size_t)h * dk + c) = __floats2half2_rn(v[0], v[1]);
    }
}

constexpr int MAX_SPLITS = 128;
constexpr int VR = 4;          // value rows of a warp of latent_merge
constexpr int BATCH = 8;       // splits whose sums are under way together

// Column group `col` (four columns) of a head's split sums: those of splits first, first + step, ... added up under a common maximum.
__device__ __forceinline__ void add_splits(const float* acc, const float2* ml, int splits, int cp, int col, int first, int step, float4& o, float& m, float& l) {
    o = make_float4(0.f, 0.f, 0.f, 0.f);
    m = -1e30f;
    l = 0.f;
    for (int s0 = first; s0 < splits; s0 += step * BATCH) {
        float2 st[BATCH];
        float4 v[BATCH];
#pragma unroll
        for (int i = 0; i < BATCH; i++) {
            const int s = s0 + step * i;
            st[i] = s < splits ? ml[s] : make_float2(-1e30f, 0.f);
            v[i] = s < splits && 4 * col < cp ? *(const float4*)(acc + (size_t)s * cp + 4 * col) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
        float mn = m;
#pragma unroll
        for (int i = 0; i < BATCH; i++) mn = st[i].y > 0.f ? fmaxf(mn, st[i].x) : mn;
        const float c = expf(m - mn);
        o.x *= c; o.y *= c; o.z *= c; o.w *= c;
        l *= c;
        m = mn;
#pragma unroll
        for (int i = 0; i < BATCH; i++) {
            if (!(st[i].y > 0.f)) continue;        // splits without keys leave their sums unwritten
            const float w = expf(st[i].x - mn);
            l += w * st[i].y;
            o.x += w * v[i].x; o.y += w * v[i].y; o.z += w * v[i].z; o.w += w * v[i].w;
        }
    }
}

// grid (heads, value parts of 8 VR, rows); a warp multiplies VR value rows.  The chain is latency: the value rows, which do not depend on
// the producer kernel, are in registers before the wait (rows of up to 512 16-bit values), and the split sums are requested together with
// their statistics, every other split by each half of the CTA.
template <typename WT>
__global__ void __launch_bounds__(256) latent_merge_kernel(const __grid_constant__ LatentMergeArgs a) {
    constexpr bool PRE = sizeof(WT) == 2;
    extern __shared__ __align__(16) float so[];    // [cp], then the second half's sums [cp]
    __shared__ float s_m[2], s_l[2];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.x, i = blockIdx.z;
    const int v0 = (blockIdx.y * 8 + warp) * VR;
    const WT* uv = (const WT*)a.uv + ((size_t)h * a.vdim + v0) * a.cp;
    const bool pre = PRE && a.cp <= 512;
    uint4 wv[PRE ? VR : 1][2];
    pdl_launch();
    if (pre) {
#pragma unroll
        for (int j = 0; j < VR; j++)
#pragma unroll
            for (int u = 0; u < 2; u++) {
                const int c = 8 * lane + 256 * u;
                wv[PRE ? j : 0][u] = v0 + j < a.vdim && c < a.cp ? ldg16(uv + (size_t)j * a.cp + c) : make_uint4(0, 0, 0, 0);
            }
    } else {
        for (int j = 0; j < VR; j++)
            if (v0 + j < a.vdim)
                for (int c = lane * (128 / (int)sizeof(WT)); c < a.cp; c += 32 * (128 / (int)sizeof(WT)))
                    asm volatile("prefetch.global.L2 [%0];" ::"l"(uv + (size_t)j * a.cp + c));
    }
    pdl_wait();
    const float* acc = a.acc + ((size_t)i * a.n_heads + h) * a.splits * a.cp;
    if (a.ml) {
        const float2* ml = a.ml + ((size_t)i * a.n_heads + h) * a.splits;
        const int part = tid >> 7;
        float4 o;
        float m, l;
        for (int c0 = 0; c0 < a.cp; c0 += 512) {   // one turn for latents of up to 512 values
            const int c = c0 + 4 * (tid & 127);
            add_splits(acc, ml, a.splits, a.cp, c >> 2, part, 2, o, m, l);
            if (c < a.cp) *(float4*)(so + part * a.cp + c) = o;
            if ((tid & 127) == 0) {
                s_m[part] = m;
                s_l[part] = l;
            }
        }
        __syncthreads();
        const float mn = fmaxf(s_m[0], s_m[1]), c0 = expf(s_m[0] - mn), c1 = expf(s_m[1] - mn), inv = 1.f / (c0 * s_l[0] + c1 * s_l[1]);
        for (int c = tid; c < a.cp; c += 256) so[c] = (c0 * so[c] + c1 * so[a.cp + c]) * inv;
    } else {
        for (int c = tid; c < a.cp; c += 256) so[c] = acc[c];
    }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < VR; j++) {
        const int v = v0 + j;
        if (v >= a.vdim) return;
        float sum = 0.f;
        auto add = [&](const float (&f)[8], int c) {
            const float4 x = *(const float4*)(so + c), y = *(const float4*)(so + c + 4);
            sum += f[0] * x.x + f[1] * x.y + f[2] * x.z + f[3] * x.w + f[4] * y.x + f[5] * y.y + f[6] * y.z + f[7] * y.w;
        };
        if (pre) {
#pragma unroll
            for (int u = 0; u < 2; u++) {
                const int c = 8 * lane + 256 * u;
                const uint4 w = wv[PRE ? j : 0][u];
                const uint32_t q[4] = {w.x, w.y, w.z, w.w};
                float f[8];
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    f[2 * e] = __uint_as_float(q[e] << 16);
                    f[2 * e + 1] = __uint_as_float(q[e] & 0xffff0000u);
                }
                if (c < a.cp) add(f, c);
            }
        } else {
            for (int c = 8 * lane; c < a.cp; c += 256) {
                float f[8];
                load8<WT>(uv + (size_t)j * a.cp + c, f);
                add(f, c);
            }
        }
        sum = warp_sum(sum);
        if (lane == 0) {
            const size_t o = (size_t)(a.rows ? a.rows[i] : i) * a.ldo + (size_t)h * a.vdim + v;
            if (a.out16) ((__nv_bfloat16*)a.out)[o] = __float2bfloat16_rn(sum);
            else ((float*)a.out)[o] = sum;
        }
    }
}

// grid (heads, rows): the split sums of a head added up, as bf16 rows [row][head][cp] of `merged`
__global__ void __launch_bounds__(128) latent_reduce_kernel(const __grid_constant__ LatentMergeArgs a, __nv_bfloat16* merged) {
    const int h = blockIdx.x, i = blockIdx.y;
    pdl_launch();
    pdl_wait();
    const size_t at = (size_t)i * a.n_heads + h;
    for (int c = 4 * threadIdx.x; c < a.cp; c += 512) {
        float4 o;
        float m, l;
        add_splits(a.acc + at * a.splits * a.cp, a.ml + at * a.splits, a.splits, a.cp, c >> 2, 0, 1, o, m, l);
        const float inv = 1.f / l;
        const __nv_bfloat162 x = __floats2bfloat162_rn(o.x * inv, o.y * inv), y = __floats2bfloat162_rn(o.z * inv, o.w * inv);
        *(uint2*)(merged + at * a.cp + c) = make_uint2(*reinterpret_cast<const uint32_t*>(&x), *reinterpret_cast<const uint32_t*>(&y));
    }
}

__device__ __forceinline__ void mma_bf16(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// grid (heads, value parts of 32, row groups of 16), 4 warps; a warp multiplies 8 value rows with 16 merged rows.  Both operands run along cp, so a
// thread loads eight consecutive values of each and uses them as the fragments of two products: the order of the terms is the same on both sides.
__global__ void __launch_bounds__(128) latent_values_kernel(const __grid_constant__ LatentMergeArgs a, const __nv_bfloat16* merged, int n) {
    const int lane = threadIdx.x & 31, g = lane >> 2, tq = lane & 3, h = blockIdx.x, i0 = blockIdx.z * 16;
    const int v0 = blockIdx.y * 32 + 8 * (threadIdx.x >> 5);
    if (v0 >= a.vdim) return;
    const __nv_bfloat16* w = (const __nv_bfloat16*)a.uv + ((size_t)h * a.vdim + min(v0 + g, a.vdim - 1)) * a.cp + 8 * tq;
    const __nv_bfloat16* r0 = merged + ((size_t)min(i0 + g, n - 1) * a.n_heads + h) * a.cp + 8 * tq;
    const __nv_bfloat16* r1 = merged + ((size_t)min(i0 + g + 8, n - 1) * a.n_heads + h) * a.cp + 8 * tq;
    const uint4 zero = make_uint4(0, 0, 0, 0);
    float c[4] = {0.f, 0.f, 0.f, 0.f}, d[4] = {0.f, 0.f, 0.f, 0.f};
    pdl_launch();
    for (int k = 0; k < a.cp; k += 32) asm volatile("prefetch.global.L2 [%0];" ::"l"(w + k));
    pdl_wait();
#pragma unroll 4
    for (int k = 0; k < a.cp; k += 32) {
        const bool in = k + 8 * tq < a.cp;         // cp is a multiple of 16
        const uint4 b = in ? ldg16(w + k) : zero, x = in ? *(const uint4*)(r0 + k) : zero, y = in ? *(const uint4*)(r1 + k) : zero;
        mma_bf16(c, x.x, y.x, x.y, y.y, b.x, b.y);
        mma_bf16(d, x.z, y.z, x.w, y.w, b.z, b.w);
    }
#pragma unroll
    for (int e = 0; e < 4; e++) {
        const int i = i0 + g + 8 * (e >> 1), v = v0 + 2 * tq + (e & 1);
        if (i >= n || v >= a.vdim) continue;
        const size_t o = (size_t)(a.rows ? a.rows[i] : i) * a.ldo + (size_t)h * a.vdim + v;
        if (a.out16) ((__nv_bfloat16*)a.out)[o] = __float2bfloat16_rn(c[e] + d[e]);
        else ((float*)a.out)[o] = c[e] + d[e];
    }
}

__global__ void __launch_bounds__(256) latent_gather_kernel(const __grid_constant__ LatentGatherArgs a) {
    const int4 q = a.seqs[blockIdx.y];
    const int pos = q.w + blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (pos >= q.y) return;
    const __half* src = a.cache + paged_row(a.page_table + (size_t)q.z * a.max_pages, pos, 1, 0) * a.w;
    __nv_bfloat16* c = a.c + (size_t)(q.x + pos) * a.cp;
    for (int i = 8 * lane; i < a.cp; i += 256) {
        const uint4 v = *(const uint4*)(src + i);
        const uint32_t w[4] = {v.x, v.y, v.z, v.w};
        uint32_t o[4];
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const float2 f = __half22float2(*reinterpret_cast<const __half2*>(&w[j]));
            const __nv_bfloat162 b = __floats2bfloat162_rn(f.x, f.y);
            o[j] = *reinterpret_cast<const uint32_t*>(&b);
        }
        *(uint4*)(c + i) = make_uint4(o[0], o[1], o[2], o[3]);
    }
    __half* r = a.r + (size_t)(q.x + pos) * a.rp;
    for (int i = lane; i < a.rp; i += 32) r[i] = i < a.rot ? src[a.cp + i] : __float2half_rn(0.f);
}

template <typename CT, typename WT>
const void* step_fn(int nb) {
    return nb == 1 ? (const void*)latent_step_kernel<CT, WT, 1> : (const void*)latent_step_kernel<CT, WT, 4>;
}

}  // namespace

// Cache rows (append) and absorbed queries of n rows; without uk the query rows of the long form (f16 caches).  Returns a cudaError_t value, as do the entry points below.
B2_API int b2_latent_step(const LatentStepArgs* a, int n, int pdl, cudaStream_t st) {
    if (n < 1 || a->n_heads < 1 || a->dim < 1 || a->rot < 0 || (a->rot & 1) || a->rank < 1 || a->cp < a->rank || (a->cp & 15) || a->w < a->cp + a->rot || (a->rot && !a->freqs) ||
        !a->q_out || !a->q || !a->c || a->ldq < a->n_heads * (a->dim + a->rot) || a->ldc < a->rank + a->rot || ((uintptr_t)a->uk & 15) || (!a->uk && (a->cache32 || a->dp < a->dim || a->rp < a->rot || (a->dp & 1) || (a->rp & 1))) || a->dim > 8192 || a->max_pages < 1)
        return (int)cudaErrorInvalidValue;
    LatentStepArgs c = *a;
    void* args[] = {&c, &n};
    const size_t angles = (size_t)a->rot * 4;
    if (angles > 32 * 1024) return (int)cudaErrorNotSupported;
    if (!a->uk) return launch_rows((const void*)latent_rows_kernel, dim3(n), dim3(256), angles, args, st, pdl);
    const int nb = n == 1 ? 1 : 4, parts = (a->cp + COLS - 1) / COLS;
    const void* fn = a->cache32 ? (a->w32 ? step_fn<float, float>(nb) : step_fn<float, __nv_bfloat16>(nb)) : (a->w32 ? step_fn<__half, float>(nb) : step_fn<__half, __nv_bfloat16>(nb));
    const size_t rows = (size_t)nb * a->dim * 4, smem = rows > angles ? rows : angles;
    if (smem > 32 * 1024) return (int)cudaErrorNotSupported;
    if ((n + nb - 1) / nb > 65535) return (int)cudaErrorInvalidValue;
    return launch_rows(fn, dim3(a->n_heads * parts + nb, (n + nb - 1) / nb), dim3(256), smem, args, st, pdl);
}

// With `merged` (bf16 [n][heads][cp] of scratch) the two-launch form: 16-bit values and splits with statistics only.
B2_API int b2_latent_merge(const LatentMergeArgs* a, int n, void* merged, int pdl, cudaStream_t st) {
    if (n < 1 || n > 65535 || a->n_heads < 1 || a->splits < 1 || a->splits > MAX_SPLITS || (!a->ml && a->splits != 1) || (a->cp & 15) || a->vdim < 1 || ((uintptr_t)a->uv & 15) ||
        ((uintptr_t)a->acc & 15) || (merged && (a->w32 || !a->ml || ((uintptr_t)merged & 15))))
        return (int)cudaErrorInvalidValue;
    LatentMergeArgs c = *a;
    if (merged) {
        void* args[] = {&c, &merged, &n};
        const int rc = launch_rows((const void*)latent_reduce_kernel, dim3(a->n_heads, n), dim3(128), 0, args, st, pdl);
        if (rc) return rc;
        return launch_rows((const void*)latent_values_kernel, dim3(a->n_heads, (a->vdim + 31) / 32, (n + 15) / 16), dim3(128), 0, args, st, pdl);
    }
    const size_t smem = (size_t)2 * a->cp * 4;
    if (smem > 40 * 1024) return (int)cudaErrorNotSupported;
    void* args[] = {&c};
    return launch_rows(a->w32 ? (const void*)latent_merge_kernel<float> : (const void*)latent_merge_kernel<__nv_bfloat16>, dim3(a->n_heads, (a->vdim + 8 * VR - 1) / (8 * VR), n),
                       dim3(256), smem, args, st, pdl);
}

B2_API int b2_latent_gather(const LatentGatherArgs* a, int n_seqs, int max_len, cudaStream_t st) {
    if (n_seqs < 1 || n_seqs > 65535 || max_len < 1 || (a->cp & 15) || (a->w & 7) || a->rp < a->rot) return (int)cudaErrorInvalidValue;
    latent_gather_kernel<<<dim3((max_len + 7) / 8, n_seqs), 256, 0, st>>>(*a);
    return (int)cudaGetLastError();
}
