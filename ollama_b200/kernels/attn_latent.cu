// Split-K attention of query rows in the latent space over a paged latent cache (latent.cu), sm_100a.
//
// All heads of a row score the same cache rows, so the heads are the rows of m16n8k16 tiles and a cache row is read once for up to 32
// heads: score = q . (latent | rotated part), result = sum of p times the latent part of the same row.  grid = (splits, groups of heads,
// query rows), 8 warps.  Tiles of 64 positions (a page) arrive by cp.async in NS stages.  Per tile each warp scores 8 positions, the
// soft-max statistics of a head are kept by a few neighbouring threads, and each warp owns 16-column units of the result.
#include "rows.cuh"

struct LatentAttnArgs {
    const __half* q;         // [n][heads][w]
    const __half* cache;     // [pages][64][w]
    const int* rows;         // step rows of the n queries, or null
    const int* positions;    // of the step's rows
    const int* slots;
    const int* page_table;   // [slots][max_pages]
    int max_pages;
    int n_heads, cp, w, splits;
    float scale;
    float* acc;              // [n][heads][splits][cp]; not written for splits without positions
    float2* ml;              // [n][heads][splits]
};

namespace {

constexpr int BN = 64, PAD = 8, LDS = BN + 4, LDP = BN + 8;

__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_f16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_addr(dst)), "l"(src) : "memory");
}

// MT: tiles of 16 heads per CTA; NU: 16-column units of the result per warp
template <int MT, int NU, int NS>
__global__ void __launch_bounds__(256) attn_latent_kernel(const __grid_constant__ LatentAttnArgs a) {
    constexpr int HR = 16 * MT, TPR = 256 / HR, KPT = BN / TPR;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __shared__ float s_corr[HR];
    const int ld = a.w + PAD;
    __half* sQ = reinterpret_cast<__half*>(smem_raw);            // [HR][ld]
    __half* sKV = sQ + HR * ld;                                  // [NS][BN][ld]
    float* sS = reinterpret_cast<float*>(sKV + NS * BN * ld);    // [HR][LDS]
    __half* sP = reinterpret_cast<__half*>(sS + HR * LDS);       // [HR][LDP]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
    const int split = blockIdx.x, head0 = blockIdx.y * HR, i = blockIdx.z;
    const int heads = min(HR, a.n_heads - head0), chunks = a.w >> 3;

    pdl_launch();
    pdl_wait();
    const int row = a.rows ? a.rows[i] : i;
    const int kv_len = a.positions[row] + 1;
    const int* table = a.page_table + (size_t)a.slots[row] * a.max_pages;
    const int pages = (kv_len + BN - 1) / BN, per = (pages + a.splits - 1) / a.splits;
    const int t0 = split * per, n_tiles = min(per, pages - t0);
    if (n_tiles <= 0) {
        for (int h = tid; h < heads; h += 256) a.ml[((size_t)i * a.n_heads + head0 + h) * a.splits + split] = make_float2(-1e30f, 0.f);
        return;
    }
    auto load_tile = [&](int tile) {
        const __half* src = a.cache + paged_row(table, (t0 + tile) * BN, 1, 0) * a.w;
        __half* dst = sKV + (tile % NS) * BN * ld;
        for (int c = tid; c < BN * chunks; c += 256) {
            const int r = c / chunks, col = (c - r * chunks) * 8;
            cp_async16(dst + r * ld + col, src + (size_t)r * a.w + col);
        }
    };
#pragma unroll
    for (int t = 0; t < NS - 1; t++) {
        if (t < n_tiles) load_tile(t);
        asm volatile("cp.async.commit_group;" ::: "memory");
    }
    for (int c = tid; c < HR * chunks; c += 256) {
        const int r = c / chunks, col = (c - r * chunks) * 8;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (r < heads) v = *(const uint4*)(a.q + ((size_t)i * a.n_heads + head0 + r) * a.w + col);
        *(uint4*)(sQ + r * ld + col) = v;
    }
    float o[MT][NU][2][4];
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
        for (int u = 0; u < NU; u++)
#pragma unroll
            for (int j = 0; j < 2; j++) o[m][u][j][0] = o[m][u][j][1] = o[m][u][j][2] = o[m][u][j][3] = 0.f;
    const int srow = tid / TPR, sub = tid % TPR;                 // soft-max phase: head row and first position of this thread
    float m_run = -1e30f, l_run = 0.f;
    const int units = a.cp >> 4;
    const uint32_t qa = smem_addr(sQ + ((lane & 7) + 8 * ((lane >> 3) & 1)) * ld + 8 * (lane >> 4));

    for (int tile = 0; tile < n_tiles; tile++) {
        asm volatile("cp.async.wait_group %0;" ::"n"(NS - 2) : "memory");
        __syncthreads();                                         // the tile is there; everyone has left the stage of tile - 1
        if (tile + NS - 1 < n_tiles) load_tile(tile + NS - 1);
        asm volatile("cp.async.commit_group;" ::: "memory");
        const __half* kv = sKV + (tile % NS) * BN * ld;
        float s[MT][2][4];
#pragma unroll
        for (int m = 0; m < MT; m++)
#pragma unroll
            for (int j = 0; j < 2; j++) s[m][j][0] = s[m][j][1] = s[m][j][2] = s[m][j][3] = 0.f;
        const uint32_t ka = smem_addr(kv + (8 * warp + (lane & 7)) * ld + 8 * (lane >> 3));
#pragma unroll 3
        for (int kk = 0; kk < a.w; kk += 32) {
            uint32_t kb[4];
            ldmatrix_x4(kb, ka + 2 * kk);
#pragma unroll
            for (int m = 0; m < MT; m++) {
                uint32_t q0[4], q1[4];
                ldmatrix_x4(q0, qa + 2 * (16 * m * ld + kk));
                ldmatrix_x4(q1, qa + 2 * (16 * m * ld + kk + 16));
                mma_f16(s[m][0], q0, kb[0], kb[1]);
                mma_f16(s[m][1], q1, kb[2], kb[3]);
            }
        }
#pragma unroll
        for (int m = 0; m < MT; m++) {
            float* d = sS + (16 * m + g) * LDS + 8 * warp + 2 * tq;
            *(float2*)d = make_float2(s[m][0][0] + s[m][1][0], s[m][0][1] + s[m][1][1]);
            *(float2*)(d + 8 * LDS) = make_float2(s[m][0][2] + s[m][1][2], s[m][0][3] + s[m][1][3]);
        }
        __syncthreads();
        {
            float v[KPT];
            float mx = -1e30f;
            const int k0 = (t0 + tile) * BN + sub * KPT;
#pragma unroll
            for (int j = 0; j < KPT; j += 4) {
                const float4 f = *(const float4*)(sS + srow * LDS + sub * KPT + j);
                v[j] = f.x; v[j + 1] = f.y; v[j + 2] = f.z; v[j + 3] = f.w;
            }
#pragma unroll
            for (int j = 0; j < KPT; j++) {
                v[j] = k0 + j < kv_len ? v[j] * a.scale : -INFINITY;
                mx = fmaxf(mx, v[j]);
            }
#pragma unroll
            for (int x = 1; x < TPR; x <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, x));
            const float m_new = fmaxf(m_run, mx), corr = __expf(m_run - m_new);
            float ls = 0.f;
#pragma unroll
            for (int j = 0; j < KPT; j += 2) {
                const float p0 = __expf(v[j] - m_new), p1 = __expf(v[j + 1] - m_new);
                ls += p0 + p1;
                *(__half2*)(sP + srow * LDP + sub * KPT + j) = __floats2half2_rn(p0, p1);
            }
            l_run = l_run * corr + ls;
            m_run = m_new;
            if (sub == 0) s_corr[srow] = corr;
        }
        __syncthreads();
#pragma unroll
        for (int m = 0; m < MT; m++) {
            const float c0 = s_corr[16 * m + g], c1 = s_corr[16 * m + g + 8];
#pragma unroll
            for (int u = 0; u < NU; u++)
#pragma unroll
                for (int j = 0; j < 2; j++) {
                    o[m][u][j][0] *= c0; o[m][u][j][1] *= c0;
                    o[m][u][j][2] *= c1; o[m][u][j][3] *= c1;
                }
        }
#pragma unroll
        for (int kk = 0; kk < BN / 16; kk++) {
            uint32_t pa[MT][4];
#pragma unroll
            for (int m = 0; m < MT; m++) ldmatrix_x4(pa[m], smem_addr(sP + (16 * m + (lane & 7) + 8 * ((lane >> 3) & 1)) * LDP + 16 * kk + 8 * (lane >> 4)));
#pragma unroll
            for (int u = 0; u < NU; u++) {
                const int unit = warp + 8 * u;
                if (unit >= units) continue;                     // warp-uniform
                uint32_t vb[4];
                ldmatrix_x4_trans(vb, smem_addr(kv + (16 * kk + (lane & 7) + 8 * ((lane >> 3) & 1)) * ld + 16 * unit + 8 * (lane >> 4)));
#pragma unroll
                for (int m = 0; m < MT; m++) {
                    mma_f16(o[m][u][0], pa[m], vb[0], vb[1]);
                    mma_f16(o[m][u][1], pa[m], vb[2], vb[3]);
                }
            }
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
    for (int x = 1; x < TPR; x <<= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, x);
    if (sub == 0 && srow < heads) a.ml[((size_t)i * a.n_heads + head0 + srow) * a.splits + split] = make_float2(m_run, l_run);
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
            const int h = 16 * m + g + 8 * e;
            if (h >= heads) continue;
            float* dst = a.acc + (((size_t)i * a.n_heads + head0 + h) * a.splits + split) * a.cp + 2 * tq;
#pragma unroll
            for (int u = 0; u < NU; u++) {
                const int unit = warp + 8 * u;
                if (unit >= units) continue;
                *(float2*)(dst + 16 * unit) = make_float2(o[m][u][0][2 * e], o[m][u][0][2 * e + 1]);
                *(float2*)(dst + 16 * unit + 8) = make_float2(o[m][u][1][2 * e], o[m][u][1][2 * e + 1]);
            }
        }
}

constexpr size_t SMEM_MAX = 226 * 1024;

size_t smem_bytes(int mt, int ns, int w) { return (size_t)(16 * mt + ns * BN) * (w + PAD) * 2 + (size_t)16 * mt * (LDS * 4 + LDP * 2); }

template <int MT, int NU, int NS>
int launch(const LatentAttnArgs& a, int n, int pdl, cudaStream_t st) {
    static PerDeviceOnce once;
    if (once.first()) cudaFuncSetAttribute(attn_latent_kernel<MT, NU, NS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM_MAX);
    LatentAttnArgs c = a;
    void* args[] = {&c};
    return launch_rows((const void*)attn_latent_kernel<MT, NU, NS>, dim3(a.splits, (a.n_heads + 16 * MT - 1) / (16 * MT), n), dim3(256), smem_bytes(MT, NS, a.w), args, st, pdl);
}

template <int MT, int NU>
int launch_ns(const LatentAttnArgs& a, int n, int pdl, cudaStream_t st) {
    if (smem_bytes(MT, 3, a.w) <= SMEM_MAX / 2) return launch<MT, NU, 3>(a, n, pdl, st);      // two CTAs per SM
    if (smem_bytes(MT, 2, a.w) <= SMEM_MAX) return launch<MT, NU, 2>(a, n, pdl, st);
    return (int)cudaErrorNotSupported;
}

template <int MT>
int launch_nu(const LatentAttnArgs& a, int n, int pdl, cudaStream_t st) {
    if (a.cp <= 128) return launch_ns<MT, 1>(a, n, pdl, st);
    if (a.cp <= 256) return launch_ns<MT, 2>(a, n, pdl, st);
    return launch_ns<MT, 4>(a, n, pdl, st);
}

}  // namespace

// f16 cache with w % 32 == 0 and a latent of up to 512 (padded) values; other shapes: cudaErrorNotSupported, nothing launched.
B2_API int b2_attn_latent(const LatentAttnArgs* a, int n, int pdl, cudaStream_t st) {
    if (n < 1 || a->n_heads < 1 || a->splits < 1 || a->splits > 128 || a->cp < 16 || (a->cp & 15) || a->w < a->cp || a->max_pages < 1 || ((uintptr_t)a->q & 15) || ((uintptr_t)a->cache & 15))
        return (int)cudaErrorInvalidValue;
    if ((a->w & 31) || a->cp > 512 || n > 65535) return (int)cudaErrorNotSupported;
    return a->n_heads <= 16 ? launch_nu<1>(*a, n, pdl, st) : launch_nu<2>(*a, n, pdl, st);
}
