// Argument block of the kernels of the state-space mixer with one decay per head (ssd.cu, ssd_chunk.cu).
#pragma once
#include "rows.cuh"

struct SsdArgs {
    const void* u;           // [rows][ldu]: x from column 0, B of group g at off_b + g n_state, C at off_c + g n_state
    int ldu, off_b, off_c;
    const void* z;           // [rows][ldz]
    int ldz;
    const float* dt;         // [rows][lddt], before bias and softplus
    int lddt;
    const float* dt_bias;    // [heads]
    const float* a;          // [heads], negative
    const float* d;          // [heads]
    int heads, groups, vdim, n_state;
    float* state;            // [slots][heads][vdim][n_state]
    const int4* seg;         // scan: [n_seg] (first row, rows, slot, position of the first row)
    const int* slots;        // step: [rows]
    const int* positions;    // step: [rows]
    void* out;               // [rows][ldo]
    int ldo;
};

// Prompt rows of 16-bit models in chunks on the tensor cores (ssd_chunk.cu).
int ssd_chunk_launch(const SsdArgs& a, int n_seg, int pdl, cudaStream_t st);
