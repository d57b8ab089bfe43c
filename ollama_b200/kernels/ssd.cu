// State-space mixer with one decay per head (a state of vdim x n_state per head, B and C shared by the heads of a group):
//
//   dt = softplus(dt' + b),  S[p][n] <- exp(a dt) S[p][n] + dt x[p] B[n],  y[p] = sum_n S[p][n] C[n] + D x[p],  result y silu(z)
//
// A scan over prompt rows that carries the state through portions of any length (32-bit models; the 16-bit form is in ssd_chunk.cu), a decode step of one token
// per sequence, and the RMS norm of the gated result in equal parts of a row.  x, B and C come convolved and activated (ssm.cu).  Step sizes, decays, state and norm are fp32;
// the state advances as S + S expm1(a dt), which keeps the distance of a slow decay from 1 to full precision.
//
// Heads stand `vdim` columns apart (padded to a multiple of 8, pad columns zero), B and C have rows of n_state padded to a multiple of 16 per group.
// A slot's state is [head][vdim][n_state]; a sequence at position 0 takes it as zeros.
#include "ssd.cuh"

namespace {

// LPC lanes share a channel and hold SPL state dimensions each.  Time runs in tiles of TT rows staged in shared memory; eight rows are advanced before
// their partial sums over the state are reduced.
template <int LPC, int SPL>
__global__ void __launch_bounds__(128) ssd_scan_kernel(const __grid_constant__ SsdArgs a) {
    constexpr int CH = 128 / LPC, NP = LPC * SPL, TT = NP <= 128 ? 32 : 16, U = 8;
    constexpr int PER = TT * CH / 128;
    __shared__ float s_em[TT], s_dt[TT];
    __shared__ float s_dx[TT][CH], s_y[TT][CH];
    __shared__ __align__(16) float s_b[TT][NP], s_c[TT][NP];
    const int tid = threadIdx.x, ch = tid / LPC, l = tid % LPC, h = blockIdx.y, g = h / (a.heads / a.groups);
    const int c0 = blockIdx.x * CH, c = c0 + ch;
    pdl_launch();
    pdl_wait();
    const int4 sg = a.seg[blockIdx.z];
    const int row0 = sg.x, rows = sg.y, pos0 = sg.w;
    const bool live = c < a.vdim;
    float* st = a.state + (((size_t)sg.z * a.heads + h) * a.vdim + (live ? c : 0)) * a.n_state;
    float S[SPL];
#pragma unroll
    for (int i = 0; i < SPL; i++) S[i] = live && l * SPL + i < a.n_state && pos0 > 0 ? st[l * SPL + i] : 0.f;
    const float A = a.a[h], bias = a.dt_bias[h], dd = a.d[h];
    const float* u = (const float*)a.u + (size_t)row0 * a.ldu;
    const float* z = (const float*)a.z + (size_t)row0 * a.ldz + h * a.vdim;
    const float* pdt = a.dt + (size_t)row0 * a.lddt + h;
    float* out = (float*)a.out + (size_t)row0 * a.ldo + h * a.vdim;
    const int lc = tid % CH, lt = tid / CH;      // element (lt + LPC * i, lc) of a tile is this thread's to move
    const bool lok = c0 + lc < a.vdim;
    for (int t0 = 0; t0 < rows; t0 += TT) {
        if (tid < TT) {                          // rows past the end take no step
            const float dt = t0 + tid < rows ? softplus_f(pdt[(size_t)(t0 + tid) * a.lddt] + bias) : 0.f;
            s_dt[tid] = dt;
            s_em[tid] = expm1f(A * dt);
        }
        for (int e = tid; e < TT * NP; e += 128) {
            const int t = e / NP, n = e % NP;
            const bool ok = t0 + t < rows && n < a.n_state;
            const float* r = u + (size_t)(t0 + t) * a.ldu + g * a.n_state + n;
            s_b[t][n] = ok ? r[a.off_b] : 0.f;
            s_c[t][n] = ok ? r[a.off_c] : 0.f;
        }
        float x[PER];
        __syncthreads();
#pragma unroll
        for (int i = 0; i < PER; i++) {
            const int t = lt + LPC * i;
            x[i] = lok && t0 + t < rows ? u[(size_t)(t0 + t) * a.ldu + h * a.vdim + c0 + lc] : 0.f;
            s_dx[t][lc] = s_dt[t] * x[i];
        }
        __syncthreads();
#pragma unroll 1
        for (int t = 0; t < TT && t0 + t < rows; t += U) {
            float y[U];
#pragma unroll
            for (int k = 0; k < U; k++) {
                const float em = s_em[t + k], dx = s_dx[t + k][ch];
                y[k] = 0.f;
#pragma unroll
                for (int i = 0; i < SPL; i++) {
                    S[i] = fmaf(S[i], em, S[i]) + dx * s_b[t + k][l * SPL + i];
                    y[k] += S[i] * s_c[t + k][l * SPL + i];
                }
            }
            // sum over the channel's lanes, halving the rows a lane is responsible for at each exchange
            int cnt = U, mine = 0;
#pragma unroll
            for (int o = LPC / 2; o > 0; o >>= 1) {
                if (cnt > 1) {
                    cnt >>= 1;
                    const bool up = (l & o) != 0;
#pragma unroll
                    for (int k = 0; k < U / 2; k++) {
                        if (k < cnt) {
                            const float send = up ? y[k] : y[k + cnt], keep = up ? y[k + cnt] : y[k];
                            y[k] = keep + __shfl_xor_sync(0xffffffffu, send, o);
                        }
                    }
                    if (up) mine += cnt;
                } else {
                    y[0] += __shfl_xor_sync(0xffffffffu, y[0], o);
                }
            }
            s_y[t + mine][ch] = y[0];
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < PER; i++) {
            const int t = lt + LPC * i;
            if (lok && t0 + t < rows) out[(size_t)(t0 + t) * a.ldo + c0 + lc] = (s_y[t][lc] + dd * x[i]) * silu_f(z[(size_t)(t0 + t) * a.ldz + c0 + lc]);
        }
    }
    if (!live) return;
#pragma unroll
    for (int i = 0; i < SPL; i++)
        if (l * SPL + i < a.n_state) st[l * SPL + i] = S[i];
}

template <typename T>
__device__ __forceinline__ float4 load4(const T* p);
template <>
__device__ __forceinline__ float4 load4<float>(const float* p) { return *(const float4*)p; }
template <>
__device__ __forceinline__ float4 load4<__nv_bfloat16>(const __nv_bfloat16* p) {
    const uint2 q = *(const uint2*)p;
    return make_float4(__uint_as_float(q.x << 16), __uint_as_float(q.x & 0xffff0000u), __uint_as_float(q.y << 16), __uint_as_float(q.y & 0xffff0000u));
}

// One token per sequence: LPR lanes per state row, VN float4 each, RPT rows per lane group in flight.  grid (row blocks, heads, sequences)
constexpr int RPT = 4;
template <typename T, int LPR, int VN>
__global__ void __launch_bounds__(256) ssd_step_kernel(const __grid_constant__ SsdArgs a) {
    constexpr int GR = 256 / LPR;
    const int l = threadIdx.x % LPR, grp = threadIdx.x / LPR, h = blockIdx.y, b = blockIdx.z, g = h / (a.heads / a.groups);
    const float A = a.a[h], bias = a.dt_bias[h], dd = a.d[h];
    pdl_launch();
    pdl_wait();
    const int slot = a.slots[b];
    const bool fresh = a.positions[b] == 0;
    float* base = a.state + ((size_t)slot * a.heads + h) * a.vdim * a.n_state;
    const T* u = (const T*)a.u + (size_t)b * a.ldu;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    float4 S[RPT][VN], B[VN], C[VN];
    float x[RPT];
#pragma unroll
    for (int r = 0; r < RPT; r++) {
        const int p = (blockIdx.x * RPT + r) * GR + grp;
#pragma unroll
        for (int v = 0; v < VN; v++) {
            const int n = 4 * (l + LPR * v);
            S[r][v] = p < a.vdim && n < a.n_state && !fresh ? __ldcg((const float4*)(base + (size_t)p * a.n_state + n)) : zero;
        }
        x[r] = p < a.vdim ? to_f(u[h * a.vdim + p]) : 0.f;
    }
#pragma unroll
    for (int v = 0; v < VN; v++) {
        const int n = 4 * (l + LPR * v);
        B[v] = n < a.n_state ? load4(u + a.off_b + g * a.n_state + n) : zero;
        C[v] = n < a.n_state ? load4(u + a.off_c + g * a.n_state + n) : zero;
    }
    const float dt = softplus_f(a.dt[(size_t)b * a.lddt + h] + bias), em = expm1f(A * dt);
#pragma unroll
    for (int r = 0; r < RPT; r++) {
        const int p = (blockIdx.x * RPT + r) * GR + grp;
        const float dx = dt * x[r];
        float y = 0.f;
#pragma unroll
        for (int v = 0; v < VN; v++) {
            float4& s = S[r][v];
            s.x = fmaf(s.x, em, s.x) + dx * B[v].x; s.y = fmaf(s.y, em, s.y) + dx * B[v].y;
            s.z = fmaf(s.z, em, s.z) + dx * B[v].z; s.w = fmaf(s.w, em, s.w) + dx * B[v].w;
            y += s.x * C[v].x + s.y * C[v].y + s.z * C[v].z + s.w * C[v].w;
            const int n = 4 * (l + LPR * v);
            if (p < a.vdim && n < a.n_state) *(float4*)(base + (size_t)p * a.n_state + n) = s;
        }
#pragma unroll
        for (int o = LPR / 2; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
        if (l == 0 && p < a.vdim) {
            const int c = h * a.vdim + p;
            ((T*)a.out)[(size_t)b * a.ldo + c] = from_f<T>((y + dd * x[r]) * silu_f(to_f(((const T*)a.z)[(size_t)b * a.ldz + c])));
        }
    }
}

const void* pick_scan(int n, int& ch) {
    if (n <= 16) { ch = 16; return (const void*)ssd_scan_kernel<8, 2>; }
    if (n <= 32) { ch = 16; return (const void*)ssd_scan_kernel<8, 4>; }
    if (n <= 64) { ch = 8; return (const void*)ssd_scan_kernel<16, 4>; }
    if (n <= 128) { ch = 8; return (const void*)ssd_scan_kernel<16, 8>; }
    if (n <= 256) { ch = 8; return (const void*)ssd_scan_kernel<16, 16>; }
    return nullptr;
}
template <typename T>
const void* pick_step(int n, int& rows) {
    if (n <= 32) { rows = 256 / 8 * RPT; return (const void*)ssd_step_kernel<T, 8, 1>; }
    if (n <= 64) { rows = 256 / 16 * RPT; return (const void*)ssd_step_kernel<T, 16, 1>; }
    if (n <= 128) { rows = 256 / 32 * RPT; return (const void*)ssd_step_kernel<T, 32, 1>; }
    if (n <= 256) { rows = 256 / 32 * RPT; return (const void*)ssd_step_kernel<T, 32, 2>; }
    return nullptr;
}

bool bad_ssd(const SsdArgs* a) {
    return a->heads < 1 || a->heads > 65535 || a->groups < 1 || a->heads % a->groups || a->vdim < 8 || (a->vdim & 7) || a->n_state < 16 || (a->n_state & 15) || (a->ldu & 3) || (a->off_b & 3) ||
           (a->off_c & 3) || !a->u || !a->z || !a->dt || !a->state || !a->out;
}

}  // namespace

// At most 256 state dimensions (more: cudaErrorNotSupported).  Both return a cudaError_t value.
B2_API int b2_ssd_scan(const SsdArgs* a, int n_seg, int f32, int pdl, cudaStream_t st) {
    if (n_seg < 1 || n_seg > 65535 || bad_ssd(a) || !a->seg) return (int)cudaErrorInvalidValue;
    if (!f32) return ssd_chunk_launch(*a, n_seg, pdl, st);
    int ch = 0;
    const void* fn = pick_scan(a->n_state, ch);
    if (!fn) return (int)cudaErrorNotSupported;
    SsdArgs c = *a;
    void* args[] = {&c};
    return launch_rows(fn, dim3((a->vdim + ch - 1) / ch, a->heads, n_seg), dim3(128), 0, args, st, pdl);
}

B2_API int b2_ssd_step(const SsdArgs* a, int nb, int f32, int pdl, cudaStream_t st) {
    if (nb < 1 || nb > 65535 || bad_ssd(a) || !a->slots || !a->positions) return (int)cudaErrorInvalidValue;
    int rows = 0;
    const void* fn = f32 ? pick_step<float>(a->n_state, rows) : pick_step<__nv_bfloat16>(a->n_state, rows);
    if (!fn) return (int)cudaErrorNotSupported;
    SsdArgs c = *a;
    void* args[] = {&c};
    return launch_rows(fn, dim3((a->vdim + rows - 1) / rows, a->heads, nb), dim3(256), 0, args, st, pdl);
}

// RMS norm of `groups` equal parts of every row, in place.  Rows consist of heads of vdim values, pitch vp each; parts may end inside a head.
struct GroupNormArgs {
    void* x;                 // [rows][ldx]
    int ldx, heads, vdim, vp, groups;
    const float* w;          // [heads * vp]
    float eps;
};

namespace {

// grid (rows, groups)
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) group_norm_kernel(const __grid_constant__ GroupNormArgs a) {
    __shared__ float red[8];
    const int size = a.heads * a.vdim / a.groups, i0 = blockIdx.y * size, tid = threadIdx.x;
    pdl_launch();
    pdl_wait();
    T* x = (T*)a.x + (size_t)blockIdx.x * a.ldx;
    float ss = 0.f;
    if (VEC) {
        for (int i = i0 + 4 * tid; i < i0 + size; i += 1024) {
            const float4 v = load4(x + i);
            ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
    } else {
        for (int i = i0 + tid; i < i0 + size; i += 256) {
            const float v = to_f(x[i / a.vdim * a.vp + i % a.vdim]);
            ss += v * v;
        }
    }
    ss = warp_sum(ss);
    if ((tid & 31) == 0) red[tid >> 5] = ss;
    __syncthreads();
    float total = 0.f;
#pragma unroll
    for (int i = 0; i < 8; i++) total += red[i];
    const float inv = 1.f / sqrtf(total / (float)size + a.eps);
    if (VEC) {
        for (int i = i0 + 4 * tid; i < i0 + size; i += 1024) {
            const float4 v = load4(x + i), w = __ldg((const float4*)(a.w + i));
            const float r[4] = {v.x * inv * w.x, v.y * inv * w.y, v.z * inv * w.z, v.w * inv * w.w};
            if (sizeof(T) == 2) {
                const __nv_bfloat162 lo = __floats2bfloat162_rn(r[0], r[1]), hi = __floats2bfloat162_rn(r[2], r[3]);
                *(uint2*)(x + i) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
            } else {
                *(float4*)(x + i) = make_float4(r[0], r[1], r[2], r[3]);
            }
        }
    } else {
        for (int i = i0 + tid; i < i0 + size; i += 256) {
            const int c = i / a.vdim * a.vp + i % a.vdim;
            x[c] = from_f<T>(to_f(x[c]) * inv * a.w[c]);
        }
    }
}

}  // namespace

B2_API int b2_group_norm(const GroupNormArgs* a, int rows, int f32, int pdl, cudaStream_t st) {
    if (rows < 1 || a->heads < 1 || a->vdim < 1 || a->vp < a->vdim || a->groups < 1 || a->groups > 65535 || (a->heads * a->vdim) % a->groups || a->ldx < a->heads * a->vp || !a->x || !a->w)
        return (int)cudaErrorInvalidValue;
    GroupNormArgs c = *a;
    void* args[] = {&c};
    const bool vec = a->vp == a->vdim && ((a->heads * a->vdim / a->groups) & 3) == 0 && (a->ldx & 3) == 0 && (((uintptr_t)a->x | (uintptr_t)a->w) & 15) == 0;
    const void* fn = f32 ? (vec ? (const void*)group_norm_kernel<float, true> : (const void*)group_norm_kernel<float, false>)
                         : (vec ? (const void*)group_norm_kernel<__nv_bfloat16, true> : (const void*)group_norm_kernel<__nv_bfloat16, false>);
    return launch_rows(fn, dim3(rows, a->groups), dim3(256), 0, args, st, pdl);
}
