// Choice of experts among groups of neighbours, shared by the router kernels (moe.cu, moe_rows.cu).
#pragma once
#include "common.cuh"

struct ExpertGroups {
    int count, keep;         // equal groups of neighbouring experts; only those of the `keep` best can be chosen
    float scale;             // of the weights
};

// By one warp: `s` [n] holds choice scores in shared memory.  A group is worth the sum of its two best scores; scores of groups that are not among the best (ties:
// the lower index) become -infinity.  `worth` [count] is scratch.
__device__ __forceinline__ void keep_groups(float* s, float* worth, int n, const ExpertGroups& g, int lane) {
    if (g.keep >= g.count) return;
    const int size = n / g.count;
    int sub = 1;                                   // lanes per group
    while (sub * 2 * g.count <= 32 && sub * 2 <= size) sub *= 2;
    for (int g0 = 0; g0 < g.count; g0 += 32 / sub) {
        const int q = g0 + lane / sub;
        float a = -INFINITY, b = -INFINITY;        // best and second best
        if (q < g.count) {
            for (int i = lane % sub; i < size; i += sub) {
                const float v = s[q * size + i];
                b = fmaxf(b, fminf(a, v));
                a = fmaxf(a, v);
            }
        }
        for (int o = 1; o < sub; o <<= 1) {
            const float a2 = __shfl_xor_sync(0xffffffffu, a, o), b2 = __shfl_xor_sync(0xffffffffu, b, o);
            b = fmaxf(fminf(a, a2), fmaxf(b, b2));
            a = fmaxf(a, a2);
        }
        if (q < g.count && lane % sub == 0) worth[q] = size > 1 ? a + b : a;
    }
    __syncwarp();
    for (int e = lane; e < n; e += 32) {
        const int q = e / size;
        const float w = worth[q];
        int ahead = 0;
        for (int o = 0; o < g.count; o++) ahead += worth[o] > w || (worth[o] == w && o < q);
        if (ahead >= g.keep) s[e] = -INFINITY;
    }
    __syncwarp();
}
