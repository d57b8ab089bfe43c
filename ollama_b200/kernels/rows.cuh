// Element access shared by the kernels that exist in a 16-bit and a 32-bit form.
#pragma once
#include "common.cuh"

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float to_f(__half v) { return __half2float(v); }

template <typename T>
__device__ __forceinline__ T from_f(float v);
template <>
__device__ __forceinline__ float from_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }
template <>
__device__ __forceinline__ __half from_f<__half>(float v) { return __float2half_rn(v); }

__device__ __forceinline__ float silu_f(float v) { return v / (1.f + expf(-v)); }
__device__ __forceinline__ float softplus_f(float v) { return v > 20.f ? v : log1pf(expf(v)); }

// Rotation angle of `pos` at frequency `f`, reduced to one turn: the product is formed in double, so that the angle keeps its
// 24 bits at any position.
__device__ __forceinline__ float rot_angle(int pos, double f) {
    constexpr double TURN = 6.283185307179586476925, PER_RADIAN = 1.0 / TURN;
    const double a = (double)pos * f;
    return (float)(a - TURN * rint(a * PER_RADIAN));
}

// Cache position -> row of a paged cache [page][kv head][64 positions][row length].
constexpr int PAGE_SHIFT = 6, PAGE = 1 << PAGE_SHIFT;
__device__ __forceinline__ size_t paged_row(const int* table, int pos, int n_kv_heads, int kvh) {
    return ((size_t)table[pos >> PAGE_SHIFT] * n_kv_heads + kvh) * PAGE + (pos & (PAGE - 1));
}

// Keys that the query at a position sees: not later ones, and with chunk > 0 those of its chunk of positions, with window > 0 the last `window` up to itself
// and the first `keep` of the sequence.
__device__ __forceinline__ int first_key(int pos, int chunk, int window) { return chunk > 0 ? pos - pos % chunk : window > 0 ? max(0, pos - window + 1) : 0; }
// Tiles of `tile` keys ahead of the one that holds position `first` which contain kept keys.
__device__ __forceinline__ int kept_tiles(int keep, int first, int tile) { return min((keep + tile - 1) / tile, first / tile); }

// Sigmoid gate of attention results: kind 1 one number per element, 2 one per head; before the sigmoid.
struct HeadGate {
    const float* g;          // [rows][ld]
    int ld, kind;
};
// Differential attention: a head's result is a1 - lambda a2 of its two maps, divided by its root mean square, times `scale`.
struct DiffHeads {
    float lambda, scale, eps;
    int on;
};
__device__ __forceinline__ float sigmoid_f(float v) { return __fdividef(1.f, 1.f + __expf(-v)); }
__device__ __forceinline__ float sigmoid_exact(float v) { return 1.f / (1.f + expf(-v)); }

static inline int launch_rows(const void* fn, dim3 grid, dim3 block, size_t smem, void** args, cudaStream_t st, int pdl) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute at[1];
    at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[0].val.programmaticStreamSerializationAllowed = pdl ? 1 : 0;
    cfg.attrs = at;
    cfg.numAttrs = 1;
    return (int)cudaLaunchKernelExC(&cfg, fn, args);
}

// Matrix product of a step's rows: out[m][ldo] (+)= alpha * f(a[m][lda] . b[n][ldb]^T + bias).  Served by b2_gemm_rows (bf16 operands on the
// tensor cores, gemm_tc.cu) and b2_gemm_rows_f32 (fp32 operands, gemm_f32.cu).
struct GemmRowsArgs {
    const void* a;
    const void* b;
    void* out;
    const float* bias;        // [n] or null
    // result times a table row: mul[mul_row[r] * ldm + column] in the operands' type, after the activation
    const void* mul;
    const int* mul_row;       // [m]
    // grouped over experts: b holds `experts` stacked [n][k] matrices, the rows of a are sorted by expert and every tile of 128 rows
    // belongs to expert tile_expert[row / 128] (-1: no rows)
    const int* tile_expert;
    void* copy;               // fp32 results are also stored as bf16 rows of pitch ldo here (bf16 products only), or null
    float* ws;                // scratch for splitting k (bf16 products only), or null
    long long ws_floats;
    int m, n, k, lda, ldb, ldo;
    int out_type;             // 0 fp32, 1 bf16, 2 f16
    int act;                  // out_act's number, or GLU_BASE + glu_act's: rows 2i / 2i + 1 of b are gate / up of column i
    int accumulate, experts, ldm;
    float alpha, limit;       // limit: of the clamped gated unit
    // results from column tail_col on (bias added, nothing else) go to fp32 rows of their own instead (bf16 products only), or null
    float* tail;              // [m][ld_tail]
    int tail_col, ld_tail;
    float act_p, act_q;       // numbers of the activation, where it has some
};
