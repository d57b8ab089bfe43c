// The state-space scan of ssd.cu over prompt rows of 16-bit models, on the tensor cores (mma.sync), sm_100a.
//
// Time runs in chunks of 64 rows.  With l_t the sum of a dt up to row t of the chunk and S the state before it:
//
//   y_t = exp(l_t) S C_t + sum_{s <= t} (C_t . B_s) exp(l_t - l_s) dt_s x_s + D x_t,   S <- exp(l_63) S + sum_s exp(l_63 - l_s) dt_s x_s B_s^T
//
// One CTA walks over the chunks of one head (or of a part of its columns) of one portion.  The state stays in the accumulators of its warps, fp32: warp
// (p, part) holds 16 columns times a quarter of the state dimensions, and feeds it to the products with C straight from there.  x, B and C are the 16-bit values that the
// convolution left; the fp32 factors of the products (the state, the decayed scores and the decayed steps) enter as the sum of two 16-bit numbers each, which
// keeps 16 bits of them.  The results of the parts meet in shared memory, where the gate is applied.  The next chunk's rows arrive by cp.async meanwhile.
#include "ssd.cuh"

namespace {

constexpr int Q = 64, PAD = 8;

__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_addr(p)));
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_addr(p)));
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void copy16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_addr(dst)), "l"(src) : "memory");
}
// a, b as the sum of two pairs of 16-bit numbers
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xffff0000u));
    lo = *reinterpret_cast<const uint32_t*>(&l);
}

// MT tiles of 16 columns, NP state dimensions (padded)
template <int MT, int NP>
struct Lay {
    static constexpr int SP = NP >= 64 ? 4 : 2;                             // parts of the state dimensions
    static constexpr int LX = 16 * MT + PAD, LN = NP + PAD, LM = Q + PAD, LY = 16 * MT + 4;
    static constexpr int X = Q * LX * 2, BC = Q * LN * 2;                   // bytes of one stage
    static constexpr int OFF_B = 2 * X, OFF_C = OFF_B + 2 * BC, OFF_XH = OFF_C + 2 * BC, OFF_XL = OFF_XH + X, OFF_MH = OFF_XL + X, OFF_ML = OFF_MH + Q * LM * 2,
                         OFF_Y = OFF_ML + Q * LM * 2, OFF_T = OFF_Y + SP * Q * LY * 4, TOTAL = OFF_T + 2 * 4 * Q * 4;
};

template <int MT, int NP>
__global__ void __launch_bounds__(32 * MT * Lay<MT, NP>::SP, 1) ssd_chunk_kernel(const __grid_constant__ SsdArgs a) {
    using L = Lay<MT, NP>;
    constexpr int SP = L::SP, WARPS = MT * SP, THREADS = 32 * WARPS, PT = 16 * MT, NT = NP / 8 / SP;      // NT: accumulator tiles of 8 state dimensions per warp
    constexpr int ITEMS = Q * PT / 8 / THREADS;                               // 16-byte pieces of a column tile per thread
    typedef __nv_bfloat16 bf;
    extern __shared__ __align__(16) uint8_t sm[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
    const int pt = warp % MT, part = warp / MT, h = blockIdx.y, grp = h / (a.heads / a.groups), p0 = blockIdx.x * PT, np = min(PT, a.vdim - p0);
    bf *sXh = (bf*)(sm + L::OFF_XH), *sXl = (bf*)(sm + L::OFF_XL), *sMh = (bf*)(sm + L::OFF_MH), *sMl = (bf*)(sm + L::OFF_ML);
    float *sY = (float*)(sm + L::OFF_Y), *sT = (float*)(sm + L::OFF_T);
    pdl_launch();
    for (int i = tid; i < L::OFF_XH / 16; i += THREADS) ((uint4*)sm)[i] = make_uint4(0, 0, 0, 0);      // what loads never reach stays zero
    const float A = a.a[h], bias = a.dt_bias[h], dd = a.d[h];
    pdl_wait();
    const int4 sg = a.seg[blockIdx.z];
    const int row0 = sg.x, rows = sg.y, n_chunks = (rows + Q - 1) / Q;
    const bf* u = (const bf*)a.u + (size_t)row0 * a.ldu;
    const bf* z = (const bf*)a.z + (size_t)row0 * a.ldz + h * a.vdim + p0;
    bf* out = (bf*)a.out + (size_t)row0 * a.ldo + h * a.vdim + p0;
    const int x8 = np >> 3, n8 = a.n_state >> 3;
    __syncthreads();

    auto request = [&](int c) {             // rows behind the portion's end repeat its last one; their steps are zero
        bf* x = (bf*)(sm + (c & 1) * L::X);
        bf* b = (bf*)(sm + L::OFF_B + (c & 1) * L::BC);
        bf* cc = (bf*)(sm + L::OFF_C + (c & 1) * L::BC);
        for (int i = tid; i < Q * (PT / 8); i += THREADS) {
            const int r = i / (PT / 8), k = i % (PT / 8);
            if (k < x8) copy16(x + r * L::LX + 8 * k, u + (size_t)min(c * Q + r, rows - 1) * a.ldu + h * a.vdim + p0 + 8 * k);
        }
        for (int i = tid; i < Q * (NP / 8); i += THREADS) {
            const int r = i / (NP / 8), k = i % (NP / 8);
            if (k < n8) {
                const bf* src = u + (size_t)min(c * Q + r, rows - 1) * a.ldu + grp * a.n_state + 8 * k;
                copy16(b + r * L::LN + 8 * k, src + a.off_b);
                copy16(cc + r * L::LN + 8 * k, src + a.off_c);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    // per row of chunk c: l, dt, exp(l), exp(l_63 - l) dt; by one warp, two rows a lane, whose inputs it has fetched a chunk ahead
    constexpr int STEP_WARP = WARPS == 16 ? 12 : WARPS - 1;              // of 16 warps one that has no block of scores
    float raw[2];
    auto fetch_steps = [&](int c) {
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const int r = min(c * Q + 2 * lane + i, rows - 1);
            raw[i] = a.dt[(size_t)(row0 + r) * a.lddt + h];
        }
    };
    auto steps = [&](int c) {
        float* t = sT + (c & 1) * 4 * Q;
        float dt[2], l[2];
#pragma unroll
        for (int i = 0; i < 2; i++) {
            dt[i] = c * Q + 2 * lane + i < rows ? softplus_f(raw[i] + bias) : 0.f;
            l[i] = A * dt[i];
        }
        float s = l[0] + l[1];
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float v = __shfl_up_sync(0xffffffffu, s, o);
            if (lane >= o) s += v;
        }
        const float end = __shfl_sync(0xffffffffu, s, 31);
        l[0] += s - (l[0] + l[1]);          // what the lanes before sum to
        l[1] = s;
#pragma unroll
        for (int i = 0; i < 2; i++) {
            t[2 * lane + i] = l[i];
            t[Q + 2 * lane + i] = dt[i];
            t[2 * Q + 2 * lane + i] = expf(l[i]);
            t[3 * Q + 2 * lane + i] = expf(end - l[i]) * dt[i];
        }
    };

    request(0);
    if (warp == STEP_WARP) {
        fetch_steps(0);
        steps(0);
        fetch_steps(1);
    }
    // this warp's part of the state: columns p0 + 16 pt + (g, g + 8), dimensions part * NP / SP + 8 j + 2 tq + (0, 1)
    float S[NT][4];
    float* st = a.state + (((size_t)sg.z * a.heads + h) * a.vdim + p0) * a.n_state;
    const int pr = 16 * pt + g, nc = part * (NP / SP) + 2 * tq;
#pragma unroll
    for (int j = 0; j < NT; j++)
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const bool ok = sg.w > 0 && pr + 8 * i < np && nc + 8 * j < a.n_state;
            const float2 v = ok ? *(const float2*)(st + (size_t)(pr + 8 * i) * a.n_state + nc + 8 * j) : make_float2(0.f, 0.f);
            S[j][2 * i] = v.x;
            S[j][2 * i + 1] = v.y;
        }

    const int rK = (lane & 7) + 8 * (lane >> 4), cK = 8 * ((lane >> 3) & 1);      // ldmatrix rows / columns: B operands stored [n][k], transposed A operands stored [k][m]
    const int rV = (lane & 7) + 8 * ((lane >> 3) & 1), cV = 8 * (lane >> 4);      // A operands stored [m][k], B operands stored [k][n] (transposed)
    for (int c = 0; c < n_chunks; c++) {
        const bf* sX = (const bf*)(sm + (c & 1) * L::X);
        const bf* sB = (const bf*)(sm + L::OFF_B + (c & 1) * L::BC);
        const bf* sC = (const bf*)(sm + L::OFF_C + (c & 1) * L::BC);
        const float *tl = sT + (c & 1) * 4 * Q, *tdt = tl + Q, *te = tl + 2 * Q, *tw = tl + 3 * Q;
        uint4 zv[ITEMS];
#pragma unroll
        for (int i = 0; i < ITEMS; i++) {
            const int e = tid + THREADS * i, r = c * Q + e / (PT / 8), k = e % (PT / 8);
            zv[i] = r < rows && k < x8 ? *(const uint4*)(z + (size_t)r * a.ldz + 8 * k) : make_uint4(0, 0, 0, 0);
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                     // chunk c has arrived, its predecessor is done with
        if (c + 1 < n_chunks) {
            request(c + 1);
            if (warp == STEP_WARP) {
                steps(c + 1);
                fetch_steps(c + 2);
            }
        }
        // decayed scores of blocks of 16 rows t and 16 rows s
#pragma unroll
        for (int w = warp; w < 16; w += WARPS) {
            const int tt = w & 3, b = w >> 2;
            if (b <= tt) {
                float m[2][4] = {};
#pragma unroll
                for (int kk = 0; kk < NP / 16; kk++) {
                    uint32_t ca[4], bb[4];
                    ldsm4(ca, sC + (16 * tt + rV) * L::LN + 16 * kk + cV);
                    ldsm4(bb, sB + (16 * b + rK) * L::LN + 16 * kk + cK);
                    mma(m[0], ca, bb[0], bb[1]);
                    mma(m[1], ca, bb[2], bb[3]);
                }
#pragma unroll
                for (int j = 0; j < 2; j++)
#pragma unroll
                    for (int k = 0; k < 2; k++) {
                        const int t = 16 * tt + g + 8 * k, s = 16 * b + 8 * j + 2 * tq;
                        const float lt = tl[t];
                        const float v0 = s <= t ? m[j][2 * k] * expf(lt - tl[s]) * tdt[s] : 0.f, v1 = s + 1 <= t ? m[j][2 * k + 1] * expf(lt - tl[s + 1]) * tdt[s + 1] : 0.f;
                        uint32_t hi, lo;
                        split2(v0, v1, hi, lo);
                        *(uint32_t*)(sMh + t * L::LM + s) = hi;
                        *(uint32_t*)(sMl + t * L::LM + s) = lo;
                    }
            }
        }
        // decayed steps times x
#pragma unroll
        for (int i = 0; i < ITEMS; i++) {
            const int e = tid + THREADS * i, r = e / (PT / 8), k = 8 * (e % (PT / 8));
            const uint4 v = *(const uint4*)(sX + r * L::LX + k);
            const uint32_t q[4] = {v.x, v.y, v.z, v.w};
            const float w = tw[r];
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int j = 0; j < 4; j++) split2(__uint_as_float(q[j] << 16) * w, __uint_as_float(q[j] & 0xffff0000u) * w, hi[j], lo[j]);
            *(uint4*)(sXh + r * L::LX + k) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
            *(uint4*)(sXl + r * L::LX + k) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
        }
        // y^T of all rows, over this part of the state dimensions
        float y[Q / 8][4] = {};
#pragma unroll
        for (int kk = 0; kk < NT / 2; kk++) {
            uint32_t hi[4], lo[4];
            split2(S[2 * kk][0], S[2 * kk][1], hi[0], lo[0]);
            split2(S[2 * kk][2], S[2 * kk][3], hi[1], lo[1]);
            split2(S[2 * kk + 1][0], S[2 * kk + 1][1], hi[2], lo[2]);
            split2(S[2 * kk + 1][2], S[2 * kk + 1][3], hi[3], lo[3]);
#pragma unroll
            for (int j = 0; j < Q / 8; j += 2) {
                uint32_t cb[4];
                ldsm4(cb, sC + (8 * j + rK) * L::LN + part * (NP / SP) + 16 * kk + cK);
                mma(y[j], hi, cb[0], cb[1]);
                mma(y[j + 1], hi, cb[2], cb[3]);
                mma(y[j], lo, cb[0], cb[1]);
                mma(y[j + 1], lo, cb[2], cb[3]);
            }
        }
#pragma unroll
        for (int j = 0; j < Q / 8; j++) {
            const float e0 = te[8 * j + 2 * tq], e1 = te[8 * j + 2 * tq + 1];
            y[j][0] *= e0; y[j][1] *= e1; y[j][2] *= e0; y[j][3] *= e1;
        }
        __syncthreads();                     // scores and decayed steps are there
#pragma unroll
        for (int i = 0; i < 4 / SP; i++) {
            const int b = SP == 4 ? part : part ? 1 + i : 3 * i;
            uint32_t xa[4];
            ldsm4t(xa, sX + (16 * b + rK) * L::LX + 16 * pt + cK);
#pragma unroll
            for (int j = 0; j < Q / 8; j += 2) {
                if (j < 2 * b) continue;
                uint32_t mh[4], ml[4];
                ldsm4(mh, sMh + (8 * j + rK) * L::LM + 16 * b + cK);
                ldsm4(ml, sMl + (8 * j + rK) * L::LM + 16 * b + cK);
                mma(y[j], xa, mh[0], mh[1]);
                mma(y[j + 1], xa, mh[2], mh[3]);
                mma(y[j], xa, ml[0], ml[1]);
                mma(y[j + 1], xa, ml[2], ml[3]);
            }
        }
        float* yo = sY + part * Q * L::LY + 16 * pt;
#pragma unroll
        for (int j = 0; j < Q / 8; j++) {
            const int t = 8 * j + 2 * tq;
            yo[t * L::LY + g] = y[j][0];
            yo[(t + 1) * L::LY + g] = y[j][1];
            yo[t * L::LY + g + 8] = y[j][2];
            yo[(t + 1) * L::LY + g + 8] = y[j][3];
        }
        // the state behind the chunk
        const float end = te[Q - 1];
#pragma unroll
        for (int j = 0; j < NT; j++) { S[j][0] *= end; S[j][1] *= end; S[j][2] *= end; S[j][3] *= end; }
#pragma unroll
        for (int kk = 0; kk < Q / 16; kk++) {
            uint32_t xh[4], xl[4];
            ldsm4t(xh, sXh + (16 * kk + rK) * L::LX + 16 * pt + cK);
            ldsm4t(xl, sXl + (16 * kk + rK) * L::LX + 16 * pt + cK);
#pragma unroll
            for (int j = 0; j < NT; j += 2) {
                uint32_t bb[4];
                ldsm4t(bb, sB + (16 * kk + rV) * L::LN + part * (NP / SP) + 8 * j + cV);
                mma(S[j], xh, bb[0], bb[1]);
                mma(S[j + 1], xh, bb[2], bb[3]);
                mma(S[j], xl, bb[0], bb[1]);
                mma(S[j + 1], xl, bb[2], bb[3]);
            }
        }
        __syncthreads();                     // all parts of y
#pragma unroll
        for (int i = 0; i < ITEMS; i++) {
            const int e = tid + THREADS * i, t = e / (PT / 8), k = 8 * (e % (PT / 8)), r = c * Q + t;
            if (r >= rows || k >= np) continue;
            const float* y0 = sY + t * L::LY + k;
            const uint4 v = *(const uint4*)(sX + t * L::LX + k);
            const uint32_t xq[4] = {v.x, v.y, v.z, v.w}, zq[4] = {zv[i].x, zv[i].y, zv[i].z, zv[i].w};
            uint32_t o[4];
#pragma unroll
            for (int j = 0; j < 4; j++) {
                float2 y = *(const float2*)(y0 + 2 * j);
#pragma unroll
                for (int k2 = 1; k2 < SP; k2++) {
                    const float2 q = *(const float2*)(y0 + k2 * Q * L::LY + 2 * j);
                    y.x += q.x;
                    y.y += q.y;
                }
                const float z0 = __uint_as_float(zq[j] << 16), z1 = __uint_as_float(zq[j] & 0xffff0000u);
                const float v0 = (y.x + dd * __uint_as_float(xq[j] << 16)) * z0 * sigmoid_f(z0), v1 = (y.y + dd * __uint_as_float(xq[j] & 0xffff0000u)) * z1 * sigmoid_f(z1);
                const __nv_bfloat162 b2 = __floats2bfloat162_rn(v0, v1);
                o[j] = *reinterpret_cast<const uint32_t*>(&b2);
            }
            *(uint4*)(out + (size_t)r * a.ldo + k) = make_uint4(o[0], o[1], o[2], o[3]);
        }
    }
#pragma unroll
    for (int j = 0; j < NT; j++)
#pragma unroll
        for (int i = 0; i < 2; i++)
            if (pr + 8 * i < np && nc + 8 * j < a.n_state) *(float2*)(st + (size_t)(pr + 8 * i) * a.n_state + nc + 8 * j) = make_float2(S[j][2 * i], S[j][2 * i + 1]);
}

template <int MT, int NP>
int launch(const SsdArgs& a, int n_seg, int pdl, cudaStream_t st) {
    using L = Lay<MT, NP>;
    static PerDeviceOnce once;
    if (once.first()) cudaFuncSetAttribute(ssd_chunk_kernel<MT, NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, L::TOTAL);
    SsdArgs c = a;
    void* args[] = {&c};
    return launch_rows((const void*)ssd_chunk_kernel<MT, NP>, dim3((a.vdim + 16 * MT - 1) / (16 * MT), a.heads, n_seg), dim3(32 * MT * L::SP), L::TOTAL, args, st, pdl);
}

template <int MT>
int launch_n(const SsdArgs& a, int n_seg, int pdl, cudaStream_t st) {
    if (a.n_state <= 32) return launch<MT, 32>(a, n_seg, pdl, st);
    if (a.n_state <= 64) return launch<MT, 64>(a, n_seg, pdl, st);
    if (a.n_state <= 128) return launch<MT, 128>(a, n_seg, pdl, st);
    return (int)cudaErrorNotSupported;
}

}  // namespace

int ssd_chunk_launch(const SsdArgs& a, int n_seg, int pdl, cudaStream_t st) {
    if ((a.ldu & 7) || (a.off_b & 7) || (a.off_c & 7) || (a.ldz & 7) || (a.ldo & 7) || (((uintptr_t)a.u | (uintptr_t)a.z | (uintptr_t)a.out | (uintptr_t)a.state) & 15))
        return (int)cudaErrorInvalidValue;
    if (a.n_state > 128) return a.n_state <= 256 ? launch<2, 256>(a, n_seg, pdl, st) : (int)cudaErrorNotSupported;
    // 64 columns a CTA where that gives enough of them, else 32: the scores are formed twice then, by twice the SMs
    const long wide = (long)((a.vdim + 63) / 64) * a.heads * n_seg;
    return a.vdim > 32 && wide >= 96 ? launch_n<4>(a, n_seg, pdl, st) : launch_n<2>(a, n_seg, pdl, st);
}
