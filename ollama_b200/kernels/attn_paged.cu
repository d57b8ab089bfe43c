// Attention over a paged cache: preparation of a batch of rows, an attention kernel for any head size and for 32-bit models, and
// the entry points of the tensor-core kernels' paged forms (attn_decode_mma.cu, attn_prefill_tc.cu).
//
// Cache layout per layer run: K [page][kv head][64 positions][dk], V [page][kv head][64 positions][dv]; page_table[slot][i]
// is the page that holds positions 64 i .. 64 i + 63 of the slot.  dk and dv are the padded row lengths (pad columns are zero).
//
// Masks: see first_key in rows.cuh.
#include "attn_args.cuh"
#include "rows.cuh"

namespace {

// ---------------------------------------------------------------------------------------------------------------------
// RMS norm of q and k over their whole projections or over each head, rotary embedding, q to padded fp32 rows, k and v into the cache.
// One CTA per row.
// ---------------------------------------------------------------------------------------------------------------------
template <typename CT>
__global__ void __launch_bounds__(256) paged_append_kernel(const __grid_constant__ PagedAppendArgs a) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[2][8];
    const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int kvs = a.no_append ? 0 : a.n_kv_heads, kdim = a.maps * a.dim;      // columns of a key head
    const int nq = a.n_heads * a.dim, nk = kvs * kdim, half = a.n_rot >> 1;
    float* sq = sm;                // [nq + nk]
    float* cs = sm + nq + nk;      // [half], then sines
    float* sn = cs + half;
    pdl_launch();
    pdl_wait();
    const int pos = a.positions[t], slot = a.slots[t];
    const float* row = a.qkv + (size_t)t * a.ldq;
    float s0 = 0.f, s1 = 0.f;
    if (((nq | nk | a.ldq) & 3) == 0) {
        for (int i = 4 * tid; i < nq + nk; i += 1024) {
            const float4 v = *(const float4*)(row + i);
            *(float4*)(sq + i) = v;
            const float d = v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
            if (i < nq) s0 += d;
            else s1 += d;
        }
    } else {
        for (int i = tid; i < nq + nk; i += 256) {
            const float v = row[i];
            sq[i] = v;
            if (i < nq) s0 += v * v;
            else s1 += v * v;
        }
    }
    for (int p = tid; p < half; p += 256) {
        float s, c;
        sincosf(rot_angle(pos, a.freqs[p]), &s, &c);
        sn[p] = s * a.mscale;
        cs[p] = c * a.mscale;
    }
    s0 = warp_sum(s0);
    s1 = warp_sum(s1);
    if (lane == 0) {
        red[0][warp] = s0;
        red[1][warp] = s1;
    }
    __syncthreads();
    if (a.q_norm && a.head_norm) {
        for (int h = warp; h < a.n_heads + a.n_kv_heads; h += 8) {
            float* head = sq + h * a.dim;
            const float* w = h < a.n_heads ? a.q_norm : a.k_norm;
            float s = 0.f;
            for (int d = lane; d < a.dim; d += 32) s += head[d] * head[d];
            const float inv = 1.f / sqrtf(warp_sum(s) / (float)a.dim + a.eps);
            for (int d = lane; d < a.dim; d += 32) head[d] *= inv * __ldg(w + d);
        }
        __syncthreads();
    } else if (a.q_norm) {
        s0 = s1 = 0.f;
#pragma unroll
        for (int i = 0; i < 8; i++) {
            s0 += red[0][i];
            s1 += red[1][i];
        }
        const float iq = 1.f / sqrtf(s0 / (float)nq + a.eps), ik = 1.f / sqrtf(s1 / (float)nk + a.eps);
        for (int i = tid; i < nq; i += 256) sq[i] *= iq * __ldg(a.q_norm + i);
        for (int i = tid; i < nk; i += 256) sq[nq + i] *= ik * __ldg(a.k_norm + i);
        __syncthreads();
    }
    auto rotated = [&](const float* head, int d) -> float {
        const float x = head[d];
        if (d >= a.n_rot) return x;
        return d < half ? x * cs[d] - head[d + half] * sn[d] : x * cs[d - half] + head[d - half] * sn[d - half];
    };
    const int* table = a.page_table + (size_t)slot * a.max_pages;
    for (int h = warp; h < a.n_heads + 2 * kvs; h += 8) {          // a warp per head
        if (h < a.n_heads) {
            const float* head = sq + h * a.dim;
            float* q = a.q_out + ((size_t)t * a.n_heads + h) * a.dq;
            const int off = h % a.maps * a.dim;
            for (int d = lane; d < a.dq; d += 32) q[d] = d >= off && d < off + a.dim ? rotated(head, d - off) : 0.f;
        } else if (h < a.n_heads + kvs) {
            const int g = h - a.n_heads;
            const float* head = sq + nq + g * kdim;
            CT* k = (CT*)a.k_cache + paged_row(table, pos, a.n_kv_heads, g) * a.dk;
            for (int d = lane; d < a.dk; d += 32) {
                const int off = d < a.dim ? 0 : a.dim;      // the map's first column
                k[d] = from_f<CT>(d < kdim ? rotated(head + off, d - off) : 0.f);
            }
        } else {
            const int g = h - a.n_heads - kvs;
            const float* head = row + a.v_off + g * a.vdim;
            CT* v = (CT*)a.v_cache + paged_row(table, pos, a.n_kv_heads, g) * a.dv;
            for (int d = lane; d < a.dv; d += 32) v[d] = from_f<CT>(d < a.vdim ? head[d] : 0.f);
        }
    }
}

// ---------------------------------------------------------------------------------------------------------------------
// Any head size, fp16 or fp32 cache.  One CTA per (row, head), keys in tiles of 128: a thread scores one key, the
// softmax statistics are merged across the CTA, then the threads own value columns.  The kernel of 32-bit models, and of
// head sizes the tensor-core kernels do not take.
// ---------------------------------------------------------------------------------------------------------------------
constexpr int VCOLS = 4;      // value columns per thread; wider values take a CTA per 512

template <typename CT, typename OT>
__global__ void __launch_bounds__(128) paged_attn_kernel(const __grid_constant__ PagedAttnArgs a) {
    extern __shared__ float sq[];      // [dim]
    __shared__ float sp[128];
    __shared__ float red[2][4];
    const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, v0 = blockIdx.z * 128 * VCOLS;
    pdl_launch();
    pdl_wait();
    const int pos = a.positions[t], slot = a.slots[t], g = h / (a.n_heads / a.n_kv_heads);
    const int* table = a.page_table + (size_t)slot * a.max_pages;
    const float* q = a.q + ((size_t)t * a.n_heads + h) * a.dq;
    for (int i = tid; i < a.dim; i += 128) sq[i] = q[i];
    __syncthreads();
    const int lo = first_key(pos, a.chunk, a.window), kept = min(a.window > 0 ? a.keep : 0, lo);      // kept keys first, then the ones from lo on
    float acc[VCOLS] = {}, m = -INFINITY, l = 0.f;
    for (int k0 = kept > 0 ? 0 : lo; k0 <= pos; k0 = k0 < kept && k0 + 128 >= kept ? lo : k0 + 128) {
        const int kp = k0 + tid, last = k0 < kept ? kept - 1 : pos;
        float s = -INFINITY;
        if (kp <= last) {
            const CT* kr = (const CT*)a.k_cache + paged_row(table, kp, a.n_kv_heads, g) * a.dk;
            float d = 0.f;
            for (int i = 0; i < a.dim; i++) d = fmaf(sq[i], to_f(kr[i]), d);
            s = d * a.scale;
            if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
        }
        float mx = warp_max(s);
        if (lane == 0) red[0][warp] = mx;
        __syncthreads();
        mx = fmaxf(fmaxf(red[0][0], red[0][1]), fmaxf(red[0][2], red[0][3]));
        const float mn = fmaxf(m, mx);
        const float corr = expf(m - mn);      // the first tile always holds a visible key, so mn is finite
        const float p = expf(s - mn);
        sp[tid] = p;
        const float ps = warp_sum(p);
        if (lane == 0) red[1][warp] = ps;
        __syncthreads();
        l = l * corr + red[1][0] + red[1][1] + red[1][2] + red[1][3];
        m = mn;
        const int n = min(128, last - k0 + 1);
#pragma unroll
        for (int j = 0; j < VCOLS; j++) acc[j] *= corr;
        for (int i = 0; i < n; i++) {
            const CT* vr = (const CT*)a.v_cache + paged_row(table, k0 + i, a.n_kv_heads, g) * a.dv;
            const float w = sp[i];
#pragma unroll
            for (int j = 0; j < VCOLS; j++) {
                const int d = v0 + tid + 128 * j;
                if (d < a.vdim) acc[j] = fmaf(w, to_f(vr[d]), acc[j]);
            }
        }
        __syncthreads();
    }
    OT* o = (OT*)a.out + (size_t)t * a.ldo + h * a.vdim;
#pragma unroll
    for (int j = 0; j < VCOLS; j++) {
        const int d = v0 + tid + 128 * j;
        if (d >= a.vdim) continue;
        float v = acc[j] / l;
        if (a.gate.kind) v *= sigmoid_exact(a.gate.g[(size_t)t * a.gate.ld + (a.gate.kind == 1 ? h * a.vdim + d : h)]);
        o[d] = from_f<OT>(v);
    }
}

// Merge of the decode kernel's splits into rows of pitch ldo, heads of vdim columns (the partials' rows are padded to hd).
struct PagedCombineArgs {
    const float* part_acc;
    const float2* part_ml;
    int n_heads, n_splits, hd, vdim;
    void* out;
    int ldo, out16;
    HeadGate gate;
    DiffHeads diff;
};

// Split sums of head h of batch row b at column d; the statistics and sums of several splits are requested together.
__device__ __forceinline__ float merged_split(const PagedCombineArgs& a, int b, int h, int d) {
    constexpr int BATCH = 8;
    const size_t p0 = ((size_t)b * a.n_heads + h) * a.n_splits;
    float mn = -1e30f, o = 0.f, l = 0.f;
    for (int s0 = 0; s0 < a.n_splits; s0 += BATCH) {
        float2 ml[BATCH];
        float v[BATCH], top = mn;
#pragma unroll
        for (int i = 0; i < BATCH; i++) {
            const bool in = s0 + i < a.n_splits;
            ml[i] = in ? a.part_ml[p0 + s0 + i] : make_float2(-1e30f, 0.f);
            v[i] = in ? a.part_acc[(p0 + s0 + i) * a.hd + d] : 0.f;
        }
#pragma unroll
        for (int i = 0; i < BATCH; i++) top = fmaxf(top, ml[i].x);
        const float c = __expf(mn - top);
        o *= c;
        l *= c;
        mn = top;
#pragma unroll
        for (int i = 0; i < BATCH; i++) {
            const float w = __expf(ml[i].x - mn);
            o = fmaf(v[i], w, o);
            l = fmaf(ml[i].y, w, l);
        }
    }
    return l > 0.f ? o / l : 0.f;
}

// 128 threads, with two maps of a head 256: a half each
__global__ void __launch_bounds__(256) paged_combine_kernel(const __grid_constant__ PagedCombineArgs a) {
    const int h = blockIdx.x, b = blockIdx.y, d = threadIdx.x & 127;
    pdl_launch();
    pdl_wait();
    float v;
    if (a.diff.on) {
        __shared__ float red[4], second[128];
        const int map = threadIdx.x >> 7;
        v = d < a.vdim ? merged_split(a, b, 2 * h + map, d) : 0.f;
        if (map) second[d] = v;
        __syncthreads();
        v -= a.diff.lambda * second[d];
        if (map) v = 0.f;
        const float s = warp_sum(v * v);
        if (!map && (d & 31) == 0) red[d >> 5] = s;
        __syncthreads();
        if (map) return;
        v *= a.diff.scale / sqrtf((red[0] + red[1] + red[2] + red[3]) / (float)a.vdim + a.diff.eps);
        if (d >= a.vdim) return;
    } else {
        if (d >= a.vdim) return;
        v = merged_split(a, b, h, d);
    }
    if (a.gate.kind) v *= sigmoid_f(a.gate.g[(size_t)b * a.gate.ld + (a.gate.kind == 1 ? h * a.vdim + d : h)]);
    const size_t oi = (size_t)b * a.ldo + (size_t)h * a.vdim + d;
    if (a.out16) ((__nv_bfloat16*)a.out)[oi] = __float2bfloat16_rn(v);
    else ((float*)a.out)[oi] = v;
}

// Results of both maps of every head, [rows][H][2][vdim] fp32 -> the heads' results.  A warp per (row, head).
template <typename OT>
__global__ void __launch_bounds__(128) diff_rows_kernel(const float* x, int n, int H, int vdim, const __grid_constant__ DiffHeads f, OT* out, int ldo) {
    const int i = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    pdl_launch();
    pdl_wait();
    if (i >= n * H) return;
    const float* a = x + (size_t)i * 2 * vdim;
    OT* o = out + (size_t)(i / H) * ldo + (size_t)(i % H) * vdim;
    float s = 0.f;
    for (int d = lane; d < vdim; d += 32) {
        const float v = a[d] - f.lambda * a[vdim + d];
        s += v * v;
    }
    const float r = f.scale / sqrtf(warp_sum(s) / (float)vdim + f.eps);
    for (int d = lane; d < vdim; d += 32) o[d] = from_f<OT>((a[d] - f.lambda * a[vdim + d]) * r);
}

bool bad_gate(const HeadGate& g) { return g.kind < 0 || g.kind > 2 || (g.kind && !g.g); }

bool bad_shape(int H, int G, int dim, int vdim) { return H < 1 || G < 1 || H % G || dim < 1 || vdim < 1; }

}  // namespace

// Returns a cudaError_t value (as do the entry points below).
B2_API int b2_paged_append(const PagedAppendArgs* a, int rows, int pdl, cudaStream_t st) {
    if (a->maps < 1 || a->maps > 2 || a->n_heads % a->maps || (a->maps > 1 && a->q_norm) || (a->no_append && a->q_norm)) return (int)cudaErrorInvalidValue;
    const int kdim = a->maps * a->dim;
    if (rows < 1 || bad_shape(a->n_heads, a->n_kv_heads, a->dim, a->vdim) || a->dq < kdim || a->dk < kdim || a->dv < a->vdim || a->n_rot < 0 || a->n_rot > a->dim ||
        (a->n_rot & 1) || (a->n_rot && !a->freqs) || (!a->q_norm != !a->k_norm) || a->v_off < 0 || (!a->no_append && a->v_off + a->n_kv_heads * a->vdim > a->ldq))
        return (int)cudaErrorInvalidValue;
    const size_t smem = ((size_t)a->n_heads * a->dim + (a->no_append ? 0 : (size_t)a->n_kv_heads * kdim) + a->n_rot) * 4;
    if (smem > 200 * 1024) return (int)cudaErrorNotSupported;
    static PerDeviceOnce once;
    if (once.first()) {
        cudaFuncSetAttribute(paged_append_kernel<__half>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
        cudaFuncSetAttribute(paged_append_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    }
    PagedAppendArgs c = *a;
    void* args[] = {&c};
    return launch_rows(a->cache32 ? (const void*)paged_append_kernel<float> : (const void*)paged_append_kernel<__half>, dim3(rows), dim3(256), smem, args, st, pdl);
}

B2_API int b2_paged_attn(const PagedAttnArgs* a, int rows, int pdl, cudaStream_t st) {
    if (rows < 1 || bad_shape(a->n_heads, a->n_kv_heads, a->dim, a->vdim) || a->dim > 8192 || a->n_heads > 65535 || a->window < 0 || a->keep < 0 || bad_gate(a->gate)) return (int)cudaErrorInvalidValue;
    PagedAttnArgs c = *a;
    void* args[] = {&c};
    const void* fn = a->cache32 ? (a->out16 ? (const void*)paged_attn_kernel<float, __nv_bfloat16> : (const void*)paged_attn_kernel<float, float>)
                                : (a->out16 ? (const void*)paged_attn_kernel<__half, __nv_bfloat16> : (const void*)paged_attn_kernel<__half, float>);
    return launch_rows(fn, dim3(rows, a->n_heads, (a->vdim + 128 * VCOLS - 1) / (128 * VCOLS)), dim3(128), (size_t)a->dim * 4, args, st, pdl);
}

// Decode step over a paged f16 cache: norm and rotation of the new query and key, cache append and split-K attention in one launch,
// then the merge of the splits.  cudaErrorNotSupported (nothing launched): the caller runs b2_paged_append + b2_paged_attn.
B2_API int b2_attn_decode_paged(const AttnDecodeArgs* a, const AttnRopeArgs* r, int nb, int hd, void* out, int ldo, int out16, const HeadGate* gate, const DiffHeads* diff, int pdl,
                                cudaStream_t st) {
    if (diff->on && (r->maps != 2 || r->vdim > 128)) return (int)cudaErrorInvalidValue;
    if (!r || bad_gate(*gate) || !r->qkv || !a->page_table || bad_shape(a->n_heads, a->n_kv_heads, r->dim, r->vdim) || r->dim > hd || r->vdim > hd || nb < 1 || a->n_splits < 1)
        return (int)cudaErrorInvalidValue;
    const cudaError_t e = (cudaError_t)attn_decode_mma_rope_launch(*a, *r, nb, hd, pdl, st);
    if (e != cudaSuccess) return (int)e;
    PagedCombineArgs c{a->part_acc, a->part_ml, a->n_heads, a->n_splits, hd, r->vdim, out, ldo, out16, *gate, *diff};
    void* args[] = {&c};
    return launch_rows((const void*)paged_combine_kernel, dim3(diff->on ? a->n_heads / 2 : a->n_heads, nb), dim3(diff->on ? 256 : 128), 0, args, st, pdl);
}

// The heads' results of differential attention from those of both maps, x [rows][H][2][vdim].
B2_API int b2_diff_rows(const float* x, int rows, int H, int vdim, const DiffHeads* f, void* out, int ldo, int out16, int pdl, cudaStream_t st) {
    if (rows < 1 || H < 1 || vdim < 1 || ldo < H * vdim || !x || !out || (long long)rows * H > 0x7fffffffLL) return (int)cudaErrorInvalidValue;
    DiffHeads d = *f;
    void* args[] = {&x, &rows, &H, &vdim, &d, &out, &ldo};
    return launch_rows(out16 ? (const void*)diff_rows_kernel<__nv_bfloat16> : (const void*)diff_rows_kernel<float>, dim3((unsigned)(((long long)rows * H + 3) / 4)), dim3(128), 0,
                       args, st, pdl);
}
