// Argument block shared by the decode-attention kernels (scalar split-K kernel and tensor-core split-K kernel).
#pragma once
#include "rows.cuh"

struct AttnDecodeArgs {
    const float* q;          // [nb][H][HD]
    const __half* k_cache;   // [slots][Hkv][n_ctx][HD]
    const __half* v_cache;
    const int* positions;    // [nb] position of the query token (its K/V is already in the cache)
    const int* slots;        // [nb]
    int n_heads, n_kv_heads, n_ctx, n_splits;
    float scale, softcap;
    int window;              // 0 = full
    float* part_acc;         // scratch [nb][H][splits][HD]
    float2* part_ml;         // scratch [nb][H][splits] (max, sum)
    const __half* k_scale;   // q8_0 cache (k_cache / v_cache hold int8): [slots][Hkv][n_ctx][HD/32] scales, or null for f16
    const __half* v_scale;
    // paged cache (page_table set; tensor-core kernel only): caches are [page][Hkv][64][HD], n_ctx and the scales are not used
    const int* page_table;   // [slots][max_pages]
    int max_pages;
    int chunk;               // > 0: position p sees the keys from floor(p / chunk) * chunk on
    int keep;                // with window > 0: the first `keep` keys are seen too
};

// Optional second argument of the tensor-core kernel: with `qkv` set the kernel takes the query rows straight from the
// projection output and rotates them itself, and the CTA whose split holds the query's own position rotates the new key,
// appends key and value to the cache (f16 caches only) and uses them from shared memory, so that no rotary-embedding launch
// precedes the attention.
struct AttnRopeArgs {
    const float* qkv;        // [nb][(H + 2 Hkv) * HD] raw projections (q | k | v), or null: q comes rotated from a.q
    const float* inv_freq;   // [n_rot / 2]
    float mscale;
    int n_rot, neox;
    // paged form: heads of dim / vdim columns inside rows of pitch ldq (the cache rows are padded to HD), RMS norms over the whole
    // q and k projections or over each head (or null), rotation in the half-split order with frequencies in double
    const float* q_norm;     // [H * dim], head_norm: [dim]
    const float* k_norm;     // [Hkv * dim], head_norm: [dim]
    float eps;
    int ldq, dim, vdim;
    const double* freqs;     // [n_rot / 2]
    int head_norm;
    int v_off;               // column of the first value head
    // differential attention (maps = 2): n_heads counts maps.  A cache row holds the keys of a head's maps side by side, and the query of a map stands in the
    // map's columns of an otherwise empty row, so that both maps of a head score the same cache rows
    int maps;
    int no_append;           // key and value of this position are in the cache already (another layer's); the rows of qkv hold queries only
};

// Rows of a step over a paged cache: see attn_paged.cu.
struct PagedAppendArgs {
    const float* qkv;        // [rows][ldq]: q heads | k heads | ..., value heads from column v_off on
    int ldq, n_heads, n_kv_heads, dim, vdim;
    const float* q_norm;     // [H * dim], or null with k_norm; head_norm: [dim]
    const float* k_norm;     // [Hkv * dim]
    float eps;
    const double* freqs;     // [n_rot / 2]
    int n_rot;
    const int* positions;    // [rows]
    const int* slots;        // [rows]
    const int* page_table;   // [slots][max_pages]
    int max_pages;
    float* q_out;            // [rows][H][dq]
    int dq;
    void* k_cache;           // [pages][Hkv][64][dk]
    void* v_cache;           // [pages][Hkv][64][dv]
    int dk, dv, cache32;     // cache32: fp32 caches, else f16
    int head_norm, v_off;
    float mscale;            // factor of the rotated dimensions
    int maps;                // see AttnRopeArgs
    int no_append;
};

struct PagedAttnArgs {
    const float* q;          // [rows][H][dq]
    int dq, n_heads, n_kv_heads, dim, vdim;
    const void* k_cache;
    const void* v_cache;
    int dk, dv, cache32;
    const int* positions;
    const int* slots;
    const int* page_table;
    int max_pages, chunk;
    float scale, softcap;
    void* out;               // [rows][ldo], head h at column h * vdim
    int ldo, out16;
    int window, keep;
    HeadGate gate;
};

// Tensor-core variant (attn_decode_mma.cu): same partial outputs, so the same combine kernel follows.
// Returns cudaErrorNotSupported for shapes it does not take (head size other than 64 / 128, more than 16 query heads per KV head).
int attn_decode_mma_launch(const AttnDecodeArgs& a, int nb, int hd, int pdl, cudaStream_t st);
// The same with the rotary embedding and the cache append inside; cudaErrorNotSupported also for quantised caches and more
// than 256 rotated dimensions.
int attn_decode_mma_rope_launch(const AttnDecodeArgs& a, const AttnRopeArgs& r, int nb, int hd, int pdl, cudaStream_t st);
