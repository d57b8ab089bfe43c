// Selective state-space mixer (a diagonal recurrence per channel and state dimension with input-dependent step size):
//
//   u = silu(conv(x)),  dt = softplus(W_dt d + b),  S[c][n] <- exp(dt_c A[c][n]) S[c][n] + dt_c u_c B[n],
//   y_c = (sum_n S[c][n] C[n] + D_c u_c) * silu(z_c)
//
// Four kernels: the causal depthwise convolution of a batch of prompt rows, the scan over prompt rows, and a decode step that
// does projection of the step size, convolution, recurrence and gate of one token per sequence in one launch.  Recurrence,
// step sizes and decays are fp32.  A slot's state is [channel][state] fp32 plus the convolution's last taps - 1 inputs; a sequence at
// position 0 takes both as zeros, whatever an earlier owner of the slot left there.
//
// A is passed as log2(e) * A, so that exp(dt A) = exp2(dt A2); 32-bit models pass A itself and advance S by S * expm1(dt A), which keeps the
// distance of a slow decay from 1 to full precision (an error of an exponential near 1 adds up over the steps that a state remembers).
#include "rows.cuh"

__device__ __forceinline__ float ex2_f(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

template <bool EXACT>
__device__ __forceinline__ float decayed(float s, float x) { return EXACT ? fmaf(s, expm1f(x), s) : s * ex2_f(x); }

// rows: token rows of one step.  seg [n_seg][4] = first row, rows, slot, position of the first row.
struct SsmConvArgs {
    const void* xz;          // [rows][ldx], x in the first `inner` columns
    int ldx, inner, taps;    // inner: padded to a multiple of 8
    const float* w;          // [taps][inner]
    const float* b;          // [inner] or null
    float* state;            // [slots][taps - 1][inner], oldest first
    const int* slots;        // [rows]
    const int* positions;    // [rows]
    const int* offs;         // [rows] index of the row within its sequence's portion
    void* u;                 // [rows][ldu]
    int ldu;
    int silu;                // activation of the results
    int shift;               // decode rows (one per slot): the state is moved on by the row's input
};

// Gates of the 16-bit form: the exponential, quotient and logarithm of the special-function unit; log(1 + e) of a small e by its series,
// whose next term is below 2e-7 of the result.
__device__ __forceinline__ float silu_fast(float v) { return __fdividef(v, 1.f + ex2_f(-1.442695041f * v)); }
__device__ __forceinline__ float softplus_fast(float v) {
    const float e = ex2_f(1.442695041f * fminf(v, 20.f));
    const float small = e * (1.f - e * (0.5f - e * (1.f / 3.f - e * (0.25f - e * 0.2f))));
    const float r = e < 0.06f ? small : __logf(1.f + e);
    return v > 20.f ? v : r;
}
template <typename T>
__device__ __forceinline__ float silu_of(float v) { return sizeof(T) == 4 ? silu_f(v) : silu_fast(v); }
template <typename T>
__device__ __forceinline__ float softplus_of(float v) { return sizeof(T) == 4 ? softplus_f(v) : softplus_fast(v); }

// Input of the convolution `back` places before row r (zeros before the sequence's start), four channels from c on.
template <typename T>
__device__ __forceinline__ void conv_input(const SsmConvArgs& a, int r, int back, int c, float (&v)[4]) {
    const int off = a.offs[r];
    if (back <= off) {
        const T* p = (const T*)a.xz + (size_t)(r - back) * a.ldx + c;
        if (sizeof(T) == 2) {
            const uint2 q = *(const uint2*)p;
            v[0] = __uint_as_float(q.x << 16); v[1] = __uint_as_float(q.x & 0xffff0000u);
            v[2] = __uint_as_float(q.y << 16); v[3] = __uint_as_float(q.y & 0xffff0000u);
        } else {
            *(float4*)v = *(const float4*)p;
        }
    } else if (a.positions[r] - back >= 0) {      // before this portion: `back - off` places before its first row
        *(float4*)v = *(const float4*)(a.state + ((size_t)a.slots[r] * (a.taps - 1) + (a.taps - 1) - (back - off)) * a.inner + c);
    } else {
        v[0] = v[1] = v[2] = v[3] = 0.f;
    }
}

// A thread carries four channels down PR rows and keeps the last inputs in registers (TAPS > 0), or reads every tap (TAPS = 0: any number).
template <typename T, int TAPS>
__global__ void __launch_bounds__(128) ssm_conv_kernel(const __grid_constant__ SsmConvArgs a, int rows, int per) {
    const int c = 4 * (blockIdx.x * 128 + threadIdx.x);
    pdl_launch();
    if (c >= a.inner) return;
    const float4 bias = a.b ? *(const float4*)(a.b + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    constexpr int W = TAPS > 0 ? TAPS : 1;
    float w[W][4], win[W][4];
    if (TAPS > 0) {
#pragma unroll
        for (int j = 0; j < W; j++) *(float4*)w[j] = *(const float4*)(a.w + (size_t)j * a.inner + c);
    }
    pdl_wait();
    const int r0 = blockIdx.y * per, r1 = min(r0 + per, rows);
    auto finish = [&](int r, float (&acc)[4]) {
        T* o = (T*)a.u + (size_t)r * a.ldu + c;
#pragma unroll
        for (int i = 0; i < 4; i++) acc[i] = a.silu ? silu_of<T>(acc[i]) : acc[i];
        if (sizeof(T) == 2) {
            const __nv_bfloat162 lo = __floats2bfloat162_rn(acc[0], acc[1]), hi = __floats2bfloat162_rn(acc[2], acc[3]);
            *(uint2*)o = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
        } else {
            *(float4*)o = make_float4(acc[0], acc[1], acc[2], acc[3]);
        }
    };
    if (TAPS == 0) {
        for (int r = r0; r < r1; r++) {
            float acc[4] = {bias.x, bias.y, bias.z, bias.w};
            for (int j = 0; j < a.taps; j++) {
                float v[4];
                conv_input<T>(a, r, a.taps - 1 - j, c, v);
                const float4 wj = *(const float4*)(a.w + (size_t)j * a.inner + c);
                acc[0] += wj.x * v[0]; acc[1] += wj.y * v[1]; acc[2] += wj.z * v[2]; acc[3] += wj.w * v[3];
                if (a.shift && j > 0) *(float4*)(a.state + ((size_t)a.slots[r] * (a.taps - 1) + j - 1) * a.inner + c) = make_float4(v[0], v[1], v[2], v[3]);
            }
            finish(r, acc);
        }
        return;
    }
    // four rows at a time, their inputs requested together
    for (int q0 = r0; q0 < r1; q0 += 4) {
        float in[4][4];
        int off[4];
#pragma unroll
        for (int q = 0; q < 4; q++) {
            const int r = min(q0 + q, r1 - 1);
            off[q] = a.offs[r];
            const T* p = (const T*)a.xz + (size_t)r * a.ldx + c;
            if (sizeof(T) == 2) {
                const uint2 v = *(const uint2*)p;
                in[q][0] = __uint_as_float(v.x << 16); in[q][1] = __uint_as_float(v.x & 0xffff0000u);
                in[q][2] = __uint_as_float(v.y << 16); in[q][3] = __uint_as_float(v.y & 0xffff0000u);
            } else {
                *(float4*)in[q] = *(const float4*)p;
            }
        }
#pragma unroll
        for (int q = 0; q < 4; q++) {
            const int r = q0 + q;
            if (r >= r1) break;
            if (r == r0 || off[q] == 0) {
#pragma unroll
                for (int j = 0; j < W - 1; j++) conv_input<T>(a, r, W - 1 - j, c, win[j]);
            }
            float acc[4] = {bias.x, bias.y, bias.z, bias.w};
#pragma unroll
            for (int i = 0; i < 4; i++) {
                win[W - 1][i] = in[q][i];
#pragma unroll
                for (int j = 0; j < W; j++) acc[i] += w[j][i] * win[j][i];
#pragma unroll
                for (int j = 0; j < W - 1; j++) win[j][i] = win[j + 1][i];
            }
            if (a.shift) {
#pragma unroll
                for (int j = 0; j < W - 1; j++) *(float4*)(a.state + ((size_t)a.slots[r] * (W - 1) + j) * a.inner + c) = *(const float4*)win[j];
            }
            finish(r, acc);
        }
    }
}

template <typename T>
static const void* pick_conv(int taps) {
    switch (taps) {
        case 2: return (const void*)ssm_conv_kernel<T, 2>;
        case 3: return (const void*)ssm_conv_kernel<T, 3>;
        case 4: return (const void*)ssm_conv_kernel<T, 4>;
        default: return (const void*)ssm_conv_kernel<T, 0>;
    }
}

B2_API int b2_ssm_conv(const SsmConvArgs* a, int rows, int f32, int pdl, cudaStream_t st) {
    if (rows < 1 || a->inner < 8 || (a->inner & 7) || a->taps < 1 || a->ldx < a->inner || (a->ldx & 3) || a->ldu < a->inner || (a->ldu & 3) || rows > 65535 * 16)
        return (int)cudaErrorInvalidValue;
    SsmConvArgs c = *a;
    int per = rows >= 1024 ? 16 : rows >= 64 ? 4 : 1;
    void* args[] = {&c, &rows, &per};
    const dim3 grid((a->inner + 511) / 512, (rows + per - 1) / per);
    return launch_rows(f32 ? pick_conv<float>(a->taps) : pick_conv<__nv_bfloat16>(a->taps), grid, dim3(128), 0, args, st, pdl);
}

// The last taps - 1 inputs of every portion become its slot's state.  grid (channels / 256, portions)
struct ConvKeepArgs {
    const void* xz;          // [rows][ldx]
    int ldx, inner, taps;
    float* state;            // [slots][taps - 1][inner], oldest first
    const int4* seg;         // [n_seg] (first row, rows, slot, position of the first row)
};

template <typename T>
__global__ void __launch_bounds__(256) conv_keep_kernel(const __grid_constant__ ConvKeepArgs a) {
    const int c = blockIdx.x * 256 + threadIdx.x;
    pdl_launch();
    pdl_wait();
    if (c >= a.inner) return;
    const int4 sg = a.seg[blockIdx.y];
    float* cs = a.state + (size_t)sg.z * (a.taps - 1) * a.inner + c;
    for (int i = 0; i < a.taps - 1; i++) {
        const int src = sg.y - (a.taps - 1) + i;      // ascending: an entry is read before it is overwritten
        cs[(size_t)i * a.inner] = src >= 0 ? to_f(((const T*)a.xz)[(size_t)(sg.x + src) * a.ldx + c]) : sg.w > 0 ? cs[(size_t)(i + sg.y) * a.inner] : 0.f;
    }
}

B2_API int b2_conv_keep(const ConvKeepArgs* a, int n_seg, int f32, int pdl, cudaStream_t st) {
    if (n_seg < 1 || n_seg > 65535 || a->inner < 1 || a->taps < 2 || a->ldx < a->inner) return (int)cudaErrorInvalidValue;
    ConvKeepArgs c = *a;
    void* args[] = {&c};
    return launch_rows(f32 ? (const void*)conv_keep_kernel<float> : (const void*)conv_keep_kernel<__nv_bfloat16>, dim3((a->inner + 255) / 256, n_seg), dim3(256), 0, args, st, pdl);
}

struct SsmScanArgs {
    const void* xz;          // [rows][ldx]: x columns 0 .. inner - 1 (for the convolution state), z from column off_z
    int ldx, off_z;
    const void* u;           // [rows][ldu]
    int ldu;
    const float* dt;         // [rows][lddt] step sizes before bias and softplus
    int lddt;
    const float* bc;         // [rows][ldbc]: B at column off_b, C at column off_b + n_state
    int ldbc, off_b;
    const float* dt_bias;    // [inner]
    const float* a2;         // [inner][n_state] log2(e) * A (fp32 form: A)
    const float* d;          // [inner]
    int inner, n_state, taps;
    float* state;            // [slots][inner][n_state]
    float* conv_state;       // [slots][taps - 1][inner]
    const int4* seg;         // [n_seg] (first row, rows, slot, position of the first row)
    void* out;               // [rows][ldo]
    int ldo;
};

// LPC lanes share a channel and hold SPL state dimensions each.  Time runs in tiles of TT rows whose inputs are fetched into
// registers while the previous tile is worked on; eight rows are advanced before their partial sums over the state are reduced, so that
// the exponentials and loads of a row do not wait for another row's shuffles.
template <typename T, int LPC, int SPL>
__global__ void __launch_bounds__(128) ssm_scan_kernel(const __grid_constant__ SsmScanArgs a) {
    constexpr int CH = 128 / LPC, NP = LPC * SPL, TT = NP <= 128 ? 32 : 16, U = 8;
    constexpr int PER = TT * CH / 128, PERN = (TT * NP + 127) / 128;
    __shared__ float2 s_dt[TT][CH];          // (dt, dt * u)
    __shared__ float s_y[TT][CH];
    __shared__ __align__(16) float s_b[TT][NP], s_c[TT][NP];
    const int tid = threadIdx.x, ch = tid / LPC, l = tid % LPC;
    const int c0 = blockIdx.x * CH, c = c0 + ch;
    pdl_launch();
    pdl_wait();
    const int4 sg = a.seg[blockIdx.y];
    const int row0 = sg.x, rows = sg.y, slot = sg.z, pos0 = sg.w;
    const bool live = c < a.inner;
    float A[SPL], S[SPL];
#pragma unroll
    for (int i = 0; i < SPL; i++) {
        const int n = l * SPL + i;
        const bool ok = live && n < a.n_state;
        A[i] = ok ? a.a2[(size_t)c * a.n_state + n] : 0.f;
        S[i] = ok && pos0 > 0 ? a.state[((size_t)slot * a.inner + c) * a.n_state + n] : 0.f;
    }
    const T* xz = (const T*)a.xz;
    const int lc = tid % CH, lt = tid / CH;      // element (lt + LPC * i, lc) of a tile is this thread's to move
    const bool lok = c0 + lc < a.inner;
    const int col = lok ? c0 + lc : 0;
    const float bias = a.dt_bias[col], dd = a.d[col];
    const T* pu = (const T*)a.u + (size_t)(row0 + lt) * a.ldu + col;
    const T* pz = xz + (size_t)(row0 + lt) * a.ldx + a.off_z + col;
    const float* pdt = a.dt + (size_t)(row0 + lt) * a.lddt + col;
    T* po = (T*)a.out + (size_t)(row0 + lt) * a.ldo + col;
    const float* pb[PERN];
    bool bok[PERN];
#pragma unroll
    for (int i = 0; i < PERN; i++) {
        const int e = tid + 128 * i, t = e / NP, n = e % NP;
        bok[i] = t < TT && n < a.n_state;
        pb[i] = a.bc + (size_t)(row0 + (bok[i] ? t : 0)) * a.ldbc + a.off_b + (bok[i] ? n : 0);
    }
    float rdt[PER], ru[PER], rz[PER], rb[PERN], rc[PERN];
    auto fetch = [&](int t0) {                   // rows t0 .. t0 + TT - 1, where the pointers stand; they move on to the next tile
        const bool full = t0 + TT <= rows;
#pragma unroll
        for (int i = 0; i < PER; i++) {
            const bool ok = full || t0 + lt + LPC * i < rows;
            rdt[i] = ok ? pdt[i * LPC * a.lddt] : 0.f;
            ru[i] = ok ? to_f(pu[i * LPC * a.ldu]) : 0.f;
            rz[i] = ok ? to_f(pz[i * LPC * a.ldx]) : 0.f;
        }
#pragma unroll
        for (int i = 0; i < PERN; i++) {
            const bool ok = bok[i] && (full || t0 + (tid + 128 * i) / NP < rows);
            rb[i] = ok ? pb[i][0] : 0.f;
            rc[i] = ok ? pb[i][a.n_state] : 0.f;
            pb[i] += (size_t)TT * a.ldbc;
        }
        pdt += (size_t)TT * a.lddt;
        pu += (size_t)TT * a.ldu;
        pz += (size_t)TT * a.ldx;
    };
    fetch(0);
    for (int t0 = 0; t0 < rows; t0 += TT) {
        float z[PER], du[PER];
#pragma unroll
        for (int i = 0; i < PER; i++) {          // rows past the end take no step
            const float dt = t0 + lt + LPC * i < rows ? softplus_of<T>(rdt[i] + bias) : 0.f;
            s_dt[lt + LPC * i][lc] = make_float2(dt, dt * ru[i]);
            du[i] = dd * ru[i];
            z[i] = rz[i];
        }
#pragma unroll
        for (int i = 0; i < PERN; i++) {
            const int e = tid + 128 * i;
            if (e < TT * NP) {
                (&s_b[0][0])[e] = rb[i];
                (&s_c[0][0])[e] = rc[i];
            }
        }
        __syncthreads();
        if (t0 + TT < rows) fetch(t0 + TT);
#pragma unroll 1
        for (int t = 0; t < TT && t0 + t < rows; t += U) {
            float y[U];
#pragma unroll
            for (int k = 0; k < U; k++) {
                const float2 dv = s_dt[t + k][ch];
                y[k] = 0.f;
#pragma unroll
                for (int i = 0; i < SPL; i++) {
                    S[i] = decayed<sizeof(T) == 4>(S[i], dv.x * A[i]) + dv.y * s_b[t + k][l * SPL + i];
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
            if (lok && t0 + lt + LPC * i < rows) po[i * LPC * a.ldo] = from_f<T>((s_y[lt + LPC * i][lc] + du[i]) * silu_of<T>(z[i]));
        }
        po += (size_t)TT * a.ldo;
    }
    if (!live) return;
#pragma unroll
    for (int i = 0; i < SPL; i++) {
        const int n = l * SPL + i;
        if (n < a.n_state) a.state[((size_t)slot * a.inner + c) * a.n_state + n] = S[i];
    }
    if (l == 0) {
        float* cs = a.conv_state + (size_t)slot * (a.taps - 1) * a.inner + c;
        for (int i = 0; i < a.taps - 1; i++) {
            const int src = rows - (a.taps - 1) + i;      // ascending: an entry is read before it is overwritten
            cs[(size_t)i * a.inner] = src >= 0 ? to_f(xz[(size_t)(row0 + src) * a.ldx + c]) : pos0 > 0 ? cs[(size_t)(i + rows) * a.inner] : 0.f;
        }
    }
}

template <typename T>
static const void* pick_scan(int n, int& ch) {
    if (n <= 16) { ch = 16; return (const void*)ssm_scan_kernel<T, 8, 2>; }
    if (n <= 32) { ch = 16; return (const void*)ssm_scan_kernel<T, 8, 4>; }
    if (n <= 64) { ch = 8; return (const void*)ssm_scan_kernel<T, 16, 4>; }
    if (n <= 128) { ch = 4; return (const void*)ssm_scan_kernel<T, 32, 4>; }
    if (n <= 256) { ch = 8; return (const void*)ssm_scan_kernel<T, 16, 16>; }
    return nullptr;
}

// At most 256 state dimensions.  The outputs' padding columns are not written.  Returns a cudaError_t value.
B2_API int b2_ssm_scan(const SsmScanArgs* a, int n_seg, int f32, int pdl, cudaStream_t st) {
    if (n_seg < 1 || n_seg > 65535 || a->inner < 8 || (a->inner & 7) || a->n_state < 1 || a->taps < 1) return (int)cudaErrorInvalidValue;
    int ch = 0;
    const void* fn = f32 ? pick_scan<float>(a->n_state, ch) : pick_scan<__nv_bfloat16>(a->n_state, ch);
    if (!fn) return (int)cudaErrorNotSupported;
    SsmScanArgs c = *a;
    void* args[] = {&c};
    return launch_rows(fn, dim3((a->inner + ch - 1) / ch, n_seg), dim3(128), 0, args, st, pdl);
}

struct SsmStepArgs {
    const void* xz;          // [nb][ldx]
    int ldx, off_z, xz16;    // xz16: bf16, else fp32
    const float* conv_w;     // [taps][inner]
    const float* conv_b;
    float* conv_state;       // [slots][taps - 1][inner]
    int taps, inner, n_state;
    const float* p;          // [nb][ldp]: low-rank step-size input at column 0, B at column off_b, C at off_b + n_state
    int ldp, off_b;
    const void* w_dt;        // [inner][rank] bf16 or fp32 (rank padded to a multiple of 8, pad columns zero)
    int rank, w32;
    const float* dt;         // [nb][lddt] projected step sizes, or null: projected here from p and w_dt
    int lddt;
    const float* dt_bias;
    const float* a2;
    const float* d;
    float* state;            // [slots][inner][n_state]
    const int* slots;
    const int* positions;
    void* out;               // [nb][ldo]
    int ldo, out16;
    int exact;               // a2 holds A: see above
    const float* u;          // [nb][ldu] convolved and activated inputs, or null: formed here
    int ldu;
};

// eight lanes per channel, four channels per warp, 32 channels per CTA; grid (channel blocks, sequences)
__global__ void __launch_bounds__(256) ssm_step_kernel(const __grid_constant__ SsmStepArgs a) {
    const int lane = threadIdx.x & 31, l = lane & 7, b = blockIdx.y;
    const int c_raw = blockIdx.x * 32 + (threadIdx.x >> 3);
    const bool live = c_raw < a.inner;
    const int c = live ? c_raw : a.inner - 1;
    const float bias = a.dt_bias[c], dd = a.d[c];
    pdl_launch();
    pdl_wait();
    const int slot = a.slots[b];
    const bool fresh = a.positions[b] == 0;
    // the first 32 state dimensions are requested at once, ahead of the step size; more than 32 are worked off behind them
    constexpr int PRE = 4;
    const float* B = a.p + (size_t)b * a.ldp + a.off_b;
    const float* C = B + a.n_state;
    float* S = a.state + ((size_t)slot * a.inner + c) * a.n_state;
    const float* A = a.a2 + (size_t)c * a.n_state;
    float pS[PRE], pA[PRE], pB[PRE], pC[PRE];
#pragma unroll
    for (int i = 0; i < PRE; i++) {
        const int n = l + 8 * i;
        const bool ok = n < a.n_state;
        pS[i] = ok && !fresh ? S[n] : 0.f;
        pA[i] = ok ? A[n] : 0.f;
        pB[i] = ok ? B[n] : 0.f;
        pC[i] = ok ? C[n] : 0.f;
    }
    float dt = 0.f;
    if (a.dt) {
        dt = a.dt[(size_t)b * a.lddt + c];
    } else {
        const float* p = a.p + (size_t)b * a.ldp;
        if (a.w32) {
            const float* w = (const float*)a.w_dt + (size_t)c * a.rank;
            for (int i = 4 * l; i < a.rank; i += 32) {
                const float4 wv = *(const float4*)(w + i), pv = *(const float4*)(p + i);
                dt += wv.x * pv.x + wv.y * pv.y + wv.z * pv.z + wv.w * pv.w;
            }
        } else {
            const __nv_bfloat16* w = (const __nv_bfloat16*)a.w_dt + (size_t)c * a.rank;
#pragma unroll 4
            for (int i = 8 * l; i < a.rank; i += 64) {
                const uint4 q = ldg16(w + i);
                const float4 p0 = *(const float4*)(p + i), p1 = *(const float4*)(p + i + 4);
                dt += __uint_as_float(q.x << 16) * p0.x + __uint_as_float(q.x & 0xffff0000u) * p0.y + __uint_as_float(q.y << 16) * p0.z +
                      __uint_as_float(q.y & 0xffff0000u) * p0.w + __uint_as_float(q.z << 16) * p1.x + __uint_as_float(q.z & 0xffff0000u) * p1.y +
                      __uint_as_float(q.w << 16) * p1.z + __uint_as_float(q.w & 0xffff0000u) * p1.w;
            }
        }
#pragma unroll
        for (int o = 4; o > 0; o >>= 1) dt += __shfl_xor_sync(0xffffffffu, dt, o);
    }
    dt = softplus_f(dt + bias);
    const size_t xi = (size_t)b * a.ldx;
    auto in = [&](int col) -> float { return a.xz16 ? to_f(((const __nv_bfloat16*)a.xz)[xi + col]) : ((const float*)a.xz)[xi + col]; };
    const float x = in(c), z = in(a.off_z + c);
    float* cs = a.conv_state + (size_t)slot * (a.taps - 1) * a.inner + c;
    float u;
    if (a.u) {
        u = a.u[(size_t)b * a.ldu + c];
    } else {
        u = a.conv_b[c] + a.conv_w[(size_t)(a.taps - 1) * a.inner + c] * x;
        if (!fresh)
            for (int j = 0; j < a.taps - 1; j++) u += cs[(size_t)j * a.inner] * a.conv_w[(size_t)j * a.inner + c];
        u = silu_f(u);
    }
    float y = 0.f;
    auto advance = [&](float old, float An, float Bn) { return (a.exact ? decayed<true>(old, dt * An) : decayed<false>(old, dt * An)) + dt * u * Bn; };
#pragma unroll
    for (int i = 0; i < PRE; i++) {
        const int n = l + 8 * i;
        if (n < a.n_state) {
            const float s = advance(pS[i], pA[i], pB[i]);
            y += s * pC[i];
            if (live) S[n] = s;
        }
    }
    for (int n = l + 8 * PRE; n < a.n_state; n += 8) {
        const float s = advance(fresh ? 0.f : S[n], A[n], B[n]);
        y += s * C[n];
        if (live) S[n] = s;
    }
#pragma unroll
    for (int o = 4; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);      // also: every lane has read the convolution state by now
    if (!live || l != 0) return;
    for (int j = 0; j < a.taps - 1; j++) cs[(size_t)j * a.inner] = j + 1 < a.taps - 1 ? (fresh ? 0.f : cs[(size_t)(j + 1) * a.inner]) : x;
    const float v = (y + dd * u) * silu_f(z);
    if (a.out16) ((__nv_bfloat16*)a.out)[(size_t)b * a.ldo + c] = __float2bfloat16_rn(v);
    else ((float*)a.out)[(size_t)b * a.ldo + c] = v;
}

B2_API int b2_ssm_step(const SsmStepArgs* a, int nb, int pdl, cudaStream_t st) {
    if (nb < 1 || nb > 65535 || a->inner < 8 || (a->inner & 7) || a->n_state < 1 || a->taps < 1 || (!a->dt && (!a->w_dt || (a->rank & 7) || (a->ldp & 3))))
        return (int)cudaErrorInvalidValue;
    SsmStepArgs c = *a;
    void* args[] = {&c};
    return launch_rows((const void*)ssm_step_kernel, dim3((a->inner + 31) / 32, nb), dim3(256), 0, args, st, pdl);
}
