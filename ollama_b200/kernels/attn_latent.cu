// Split-K attention of query rows in the latent space over a paged latent cache (latent.cu), sm_100a.
//
// All heads of a row score the same cache rows, so the heads are the rows of m16n8k16 tiles and a cache row is read once for up to 32
// heads: score = q . (latent | rotated part), result = sum of p times the latent part of the same row.  grid = (splits, groups of heads,
// query rows), 8 warps.  Tiles of a page arrive by cp.async in two stages.  The query fragments stay in registers: a warp scores half of a
// tile's positions over a quarter of the row, the quarters are added by the threads that keep a head's soft-max statistics, and each
// warp owns 16-column units of the result.
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
    int window;              // > 0: a query sees the last `window` positions up to its own
    float scale;
    float* acc;              // [n][heads][splits][cp]; not written for splits without positions
    float2* ml;              // [n][heads][splits]
};

namespace {

constexpr int BN = PAGE, PAD = 8, QUARTERS = 4;

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
template <int MT>
struct Lay {
    static constexpr int HR = 16 * MT, LDS = BN + 4, LDP = BN + 8;
    static size_t bytes(int w) { return (size_t)2 * BN * (w + PAD) * 2 + (size_t)HR * (QUARTERS * LDS * 4 + LDP * 2); }
};

// MT: tiles of 16 heads per CTA; NU: 16-column units of the result per warp; KQ: 16-column steps of a quarter of the row, at most
template <int MT, int NU, int KQ>
__global__ void __launch_bounds__(256, MT == 1 ? 2 : 1) attn_latent_kernel(const __grid_constant__ LatentAttnArgs a) {
    using L = Lay<MT>;
    constexpr int HR = L::HR, LDS = L::LDS, LDP = L::LDP, TPR = 256 / HR, KPT = BN / TPR, NT = BN / 16;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __shared__ float s_corr[HR];
    const int ld = a.w + PAD;
    __half* sKV = reinterpret_cast<__half*>(smem_raw);           // [2][BN][ld]
    float* sS = reinterpret_cast<float*>(sKV + 2 * BN * ld);     // [QUARTERS][HR][LDS]
    __half* sP = reinterpret_cast<__half*>(sS + QUARTERS * HR * LDS);      // [HR][LDP]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
    const int split = blockIdx.x, head0 = blockIdx.y * HR, i = blockIdx.z;
    const int heads = min(HR, a.n_heads - head0);

    pdl_launch();
    pdl_wait();
    const int row = a.rows ? a.rows[i] : i;
    const int kv_len = a.positions[row] + 1;
    const int* table = a.page_table + (size_t)a.slots[row] * a.max_pages;
    const int lo = a.window > 0 ? max(0, kv_len - a.window) : 0, page0 = lo / PAGE;      // first visible position and its page
    const int pages = (kv_len + PAGE - 1) / PAGE - page0, per = (pages + a.splits - 1) / a.splits;
    const int p0 = (page0 + split * per) * PAGE, n_tiles = (min(kv_len - p0, per * PAGE) + BN - 1) / BN;
    if (kv_len <= p0) {
        for (int h = tid; h < heads; h += 256) a.ml[((size_t)i * a.n_heads + head0 + h) * a.splits + split] = make_float2(-1e30f, 0.f);
        return;
    }
    auto load_tile = [&](int tile) {
        const __half* src = a.cache + paged_row(table, p0 + tile * BN + warp, 1, 0) * a.w + 8 * lane;
        const __half* end = src + a.w - 8 * lane;
        uint32_t dst = smem_addr(sKV + ((tile & 1) * BN + warp) * ld + 8 * lane);
#pragma unroll
        for (int r = 0; r < BN / 8; r++, src += 8 * a.w, end += 8 * a.w, dst += 16 * ld) {      // a warp per row
#pragma unroll
            for (int c = 0; c < (KQ * QUARTERS * 16 + 255) / 256; c++)
                if (src + 256 * c < end) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst + 512 * c), "l"(src + 256 * c) : "memory");
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load_tile(0);
    // this warp's part of the scores: positions [BN / 2 * half, + BN / 2) of a tile, columns [16 k0, 16 k1) of the row
    const int quarter = warp & 3, half = warp >> 2, steps = a.w >> 4, kq = (steps + QUARTERS - 1) / QUARTERS;
    const int k0 = quarter * kq, k1 = min(k0 + kq, steps);
    uint32_t qf[MT][KQ][4];
#pragma unroll
    for (int m = 0; m < MT; m++) {
        const __half* q0 = a.q + ((size_t)i * a.n_heads + head0 + 16 * m + g) * a.w + 2 * tq;
        const bool in0 = 16 * m + g < heads, in1 = 16 * m + g + 8 < heads;
#pragma unroll
        for (int k = 0; k < KQ; k++) {
            const bool in = k0 + k < k1;
            const __half* q = q0 + 16 * (k0 + k);
            qf[m][k][0] = in && in0 ? *(const uint32_t*)q : 0u;
            qf[m][k][1] = in && in1 ? *(const uint32_t*)(q + (size_t)8 * a.w) : 0u;
            qf[m][k][2] = in && in0 ? *(const uint32_t*)(q + 8) : 0u;
            qf[m][k][3] = in && in1 ? *(const uint32_t*)(q + (size_t)8 * a.w + 8) : 0u;
        }
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

    for (int tile = 0; tile < n_tiles; tile++) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                         // the tile is there; everyone has left the stage of tile - 1
        if (tile + 1 < n_tiles) load_tile(tile + 1);
        const __half* kv = sKV + (tile & 1) * BN * ld;
        float s[MT][NT][4];
#pragma unroll
        for (int m = 0; m < MT; m++)
#pragma unroll
            for (int j = 0; j < NT; j++) s[m][j][0] = s[m][j][1] = s[m][j][2] = s[m][j][3] = 0.f;
        const uint32_t ka = smem_addr(kv + (BN / 2 * half + (lane & 7) + 8 * (lane >> 4)) * ld + 16 * k0 + 8 * ((lane >> 3) & 1));
#pragma unroll
        for (int k = 0; k < KQ; k++) {
            if (k0 + k >= k1) break;                             // warp-uniform
#pragma unroll
            for (int j = 0; j < NT / 2; j++) {                   // 16 positions
                uint32_t kb[4];
                ldmatrix_x4(kb, ka + 2 * (16 * j * ld + 16 * k));
#pragma unroll
                for (int m = 0; m < MT; m++) {
                    mma_f16(s[m][2 * j], qf[m][k], kb[0], kb[1]);
                    mma_f16(s[m][2 * j + 1], qf[m][k], kb[2], kb[3]);
                }
            }
        }
#pragma unroll
        for (int m = 0; m < MT; m++)
#pragma unroll
            for (int j = 0; j < NT; j++) {
                float* d = sS + (quarter * HR + 16 * m + g) * LDS + BN / 2 * half + 8 * j + 2 * tq;
                *(float2*)d = make_float2(s[m][j][0], s[m][j][1]);
                *(float2*)(d + 8 * LDS) = make_float2(s[m][j][2], s[m][j][3]);
            }
        __syncthreads();
        {
            float v[KPT];
            float mx = -1e30f;
            const int kp = p0 + tile * BN + sub * KPT;
#pragma unroll
            for (int j = 0; j < KPT; j += 2) {
                float2 f = make_float2(0.f, 0.f);
#pragma unroll
                for (int x = 0; x < QUARTERS; x++) {
                    const float2 t = *(const float2*)(sS + (x * HR + srow) * LDS + sub * KPT + j);
                    f.x += t.x; f.y += t.y;
                }
                v[j] = f.x; v[j + 1] = f.y;
            }
#pragma unroll
            for (int j = 0; j < KPT; j++) {
                v[j] = kp + j < kv_len && kp + j >= lo ? v[j] * a.scale : -INFINITY;
                mx = fmaxf(mx, v[j]);
            }
#pragma unroll
            for (int x = 1; x < TPR; x <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, x));
            const float m_new = fmaxf(m_run, mx), corr = __expf(m_run - m_new);
            float ls = 0.f;
#pragma unroll
            for (int j = 0; j < KPT; j += 2) {
                const float e0 = __expf(v[j] - m_new), e1 = __expf(v[j + 1] - m_new);
                ls += e0 + e1;
                *(__half2*)(sP + srow * LDP + sub * KPT + j) = __floats2half2_rn(e0, e1);
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

template <int MT, int NU, int KQ>
int launch(const LatentAttnArgs& a, int n, int pdl, cudaStream_t st) {
    const size_t smem = Lay<MT>::bytes(a.w);
    if (smem > SMEM_MAX) return (int)cudaErrorNotSupported;
    static PerDeviceOnce once;
    if (once.first()) cudaFuncSetAttribute(attn_latent_kernel<MT, NU, KQ>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM_MAX);
    LatentAttnArgs c = a;
    void* args[] = {&c};
    return launch_rows((const void*)attn_latent_kernel<MT, NU, KQ>, dim3(a.splits, (a.n_heads + 16 * MT - 1) / (16 * MT), n), dim3(256), smem, args, st, pdl);
}

template <int MT>
int launch_w(const LatentAttnArgs& a, int n, int pdl, cudaStream_t st) {
    if (a.cp <= 128 && a.w <= 256) return launch<MT, 1, 4>(a, n, pdl, st);
    if (a.cp <= 256 && a.w <= 448) return launch<MT, 2, 7>(a, n, pdl, st);
    if (a.w <= 576) return launch<MT, 4, 9>(a, n, pdl, st);
    return launch<MT, 4, 10>(a, n, pdl, st);
}

}  // namespace

// f16 cache with rows of up to 640 values, a multiple of 32, and a latent of up to 512; other shapes: cudaErrorNotSupported, nothing launched.
B2_API int b2_attn_latent(const LatentAttnArgs* a, int n, int pdl, cudaStream_t st) {
    if (n < 1 || a->n_heads < 1 || a->splits < 1 || a->splits > 128 || a->cp < 16 || (a->cp & 15) || a->w < a->cp || a->max_pages < 1 || a->window < 0 || ((uintptr_t)a->q & 15) || ((uintptr_t)a->cache & 15))
        return (int)cudaErrorInvalidValue;
    if ((a->w & 31) || a->cp > 512 || a->w > 640 || n > 65535) return (int)cudaErrorNotSupported;
    return a->n_heads <= 16 ? launch_w<1>(*a, n, pdl, st) : launch_w<2>(*a, n, pdl, st);
}
