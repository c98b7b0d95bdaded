// State-space mixers: recurrences whose state lives in fp32 device memory, one per cache line, decayed by step sizes that
// the tokens themselves choose.
//
//   selective scan (one decay per channel and state)                              S [channels, N] per line
//       S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n;    y_c = sum_n S[c, n] C_n + D_c x_c;    out = y silu(z)
//   state-space heads (one decay per head; B and C shared by the heads of a group) S [heads, N, P] per line
//       S <- exp(-exp(A_log) dt) S + dt B x^T;                  y = S^T C + D x
//
// dt = softplus(pre-activation + bias).  x (and B, C of the second kind) come out of a short causal convolution per channel
// with a bias and silu.  A row that starts at position 0 starts from zeros, any other row continues from its line's state;
// padding tokens (t >= n_new[b]) change nothing and come out as zeros.
//
// Kernels:
//   conv_silu          convolution + silu of a column range of a projection; also moves the line's convolution state (the
//                      last taps - 1 raw inputs) when one thread sees the whole step, else conv_state does it afterwards;
//                      conv_silu_strip is its form for long 16-bit steps
//   selective_scan     states of a channel split over R lanes of NS registers (two channels per thread share the loads of B and
//                      C), tokens in blocks through four shared-memory buffers (cp.async); the R partial sums of R
//                      consecutive tokens are summed by one transposing butterfly; the other half of the CTA makes the step
//                      sizes ahead of a block and applies skip term and gate behind it.  Prompts and single tokens
//   selective_step     one token per row: the low-rank product that makes the step sizes, the recurrence and the gate
//   ssd_step           one token: a thread owns four neighbouring columns of a head's state, the rows are spread over the
//                      CTA; the state is read and written once
//   ssd_scan           token by token, a column's rows split over R lanes (fp32 prompts, short steps, unusual sizes)
//   ssd_chunk          bf16 prompts in chunks of 64 tokens on mma.sync, one CTA walks the chunks of 64 (or 32) columns of a
//                      head with the fp32 state in accumulator registers.  Operands that are products of fp32 numbers (decayed
//                      scores, scaled inputs, the state) go in as the sum of two bf16 numbers, so that their relative error
//                      is 2^-17, not 2^-9
//   gate_norm          y act(z), divided by the root mean square over equal groups of columns and weighted
// This file is compiled without fast-math: the state lives for thousands of steps.
#include "common.cuh"
#include "mma_sync.cuh"

namespace {

__device__ __forceinline__ float ldf(const float* p) { return *p; }
__device__ __forceinline__ float ldf(const bf16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void stf(float* p, float v) { *p = v; }
__device__ __forceinline__ void stf(bf16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }
// 2^x; arguments here are never positive, results below 2^-126 become zero
__device__ __forceinline__ float exp2_ftz(float x) {
    float r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
    return r;
}
// e^y for y <= 0, rounded once where it is close to 1: a decay that hardly decays is applied thousands of times, and an error of
// even one unit in its last place that always points the same way would add up.  1 + y (1 + y/2 + ... + y^7/40320) there.
__device__ __forceinline__ float decay_exp(float y) {
    if (y < -0.35f) return expf(y);
    float p = fmaf(y, 1.f / 40320.f, 1.f / 5040.f);
    p = fmaf(y, p, 1.f / 720.f);
    p = fmaf(y, p, 1.f / 120.f);
    p = fmaf(y, p, 1.f / 24.f);
    p = fmaf(y, p, 1.f / 6.f);
    p = fmaf(y, p, 0.5f);
    p = fmaf(y, p, 1.f);
    return fmaf(y, p, 1.f);
}
constexpr float LOG2E = 1.4426950408889634f;
// packed fp32 arithmetic on two neighbouring states
__device__ __forceinline__ uint64_t pair2(float lo, float hi) {
    uint64_t r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ void unpair2(uint64_t v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
    uint64_t r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}

// the decays of two states in the selective scan: fp32 serving rounds it as above, 16-bit serving takes the hardware's 2^x
template <typename T>
struct ScanDecay {
    static __device__ __forceinline__ float rate(float a) { return a * LOG2E; }
    static __device__ __forceinline__ float at(float dt, float rate) { return exp2_ftz(dt * rate); }
    static __device__ __forceinline__ uint64_t at2(uint64_t dt, uint64_t rate) {
        float lo, hi;
        unpair2(mul2(dt, rate), lo, hi);
        return pair2(exp2_ftz(lo), exp2_ftz(hi));
    }
};
template <>
struct ScanDecay<float> {
    static __device__ __forceinline__ float rate(float a) { return a; }
    static __device__ __forceinline__ float at(float dt, float rate) { return decay_exp(dt * rate); }
    static __device__ __forceinline__ uint64_t at2(uint64_t dt, uint64_t rate) {
        float lo, hi;
        unpair2(mul2(dt, rate), lo, hi);
        return pair2(decay_exp(lo), decay_exp(hi));
    }
};

// The arithmetic around the recurrences.  fp32 serving takes the library functions; 16-bit serving forms built on the hardware's
// 2^x and reciprocal, whose relative errors stay near 2^-21: softplus(z) = max(z, 0) + log1p(e^-|z|) with log1p(t) = 2 atanh(t / (2 + t))
// by its odd power series (t / (2 + t) <= 1/3, next term below 1e-8 of the value)
template <typename T>
struct ScanMath {
    static __device__ __forceinline__ float softplus(float z) {
        const float t = exp2_ftz(-fabsf(z) * LOG2E);
        const float s = __fdividef(t, 2.f + t), q = s * s;
        float p = fmaf(q, 2.f / 15.f, 2.f / 13.f);
        p = fmaf(q, p, 2.f / 11.f);
        p = fmaf(q, p, 2.f / 9.f);
        p = fmaf(q, p, 2.f / 7.f);
        p = fmaf(q, p, 2.f / 5.f);
        p = fmaf(q, p, 2.f / 3.f);
        p = fmaf(q, p, 2.f);
        return fmaf(s, p, fmaxf(z, 0.f));
    }
    static __device__ __forceinline__ float sigmoid(float z) { return __fdividef(1.f, 1.f + exp2_ftz(fminf(-z * LOG2E, 100.f))); }
    static __device__ __forceinline__ float silu(float z) { return z * sigmoid(z); }
};
template <>
struct ScanMath<float> {
    static __device__ __forceinline__ float softplus(float z) { return softplus_f(z); }
    static __device__ __forceinline__ float sigmoid(float z) { return sigmoid_f(z); }
    static __device__ __forceinline__ float silu(float z) { return silu_f(z); }
};

template <int VEC>
__device__ __forceinline__ void ldv(const float* p, float* v) {
    if (VEC == 8) {
        const float4 t = *reinterpret_cast<const float4*>(p), u = *reinterpret_cast<const float4*>(p + 4);
        v[0] = t.x, v[1] = t.y, v[2] = t.z, v[3] = t.w, v[4] = u.x, v[5] = u.y, v[6] = u.z, v[7] = u.w;
    } else if (VEC == 4) {
        const float4 t = *reinterpret_cast<const float4*>(p);
        v[0] = t.x, v[1] = t.y, v[2] = t.z, v[3] = t.w;
    } else {
        v[0] = *p;
    }
}
template <int VEC>
__device__ __forceinline__ void ldv(const bf16* p, float* v) {
    if (VEC == 8) {
        unpack8(*reinterpret_cast<const bf16x8*>(p), v);
    } else if (VEC == 4) {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const bf162*>(&raw.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const bf162*>(&raw.y));
        v[0] = a.x, v[1] = a.y, v[2] = b.x, v[3] = b.y;
    } else {
        v[0] = __bfloat162float(*p);
    }
}
template <int VEC>
__device__ __forceinline__ void stv(float* p, const float* v) {
    if (VEC == 8) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
        *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
    } else if (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else *p = v[0];
}
template <int VEC>
__device__ __forceinline__ void stv(bf16* p, const float* v) {
    if (VEC == 8) {
        *reinterpret_cast<bf16x8*>(p) = pack8(v);
    } else if (VEC == 4) {
        uint2 raw;
        *reinterpret_cast<bf162*>(&raw.x) = __floats2bfloat162_rn(v[0], v[1]);
        *reinterpret_cast<bf162*>(&raw.y) = __floats2bfloat162_rn(v[2], v[3]);
        *reinterpret_cast<uint2*>(p) = raw;
    } else {
        *p = __float2bfloat16_rn(v[0]);
    }
}

// ---- short convolution ----------------------------------------------------------------------------------------------------
// VEC raw inputs (channels c ..) at step index s, which may lie before the step: then they come from the line's state (slot
// K + s holds position p0 + s), zeros before the start of the sequence
template <typename T, int VEC>
__device__ __forceinline__ void conv_input(const T* __restrict__ row0, long long ld, const float* __restrict__ st, int s, int p0,
                                           int K, int C, int c, float* v) {
    if (s >= 0) {
        ldv<VEC>(row0 + (long long)s * ld + c, v);
    } else if (p0 + s < 0) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] = 0.f;
    } else {
        ldv<VEC>(st + (long long)(K + s) * C + c, v);
    }
}

// slot s of the line's state <- raw input of position (p0 + n) - K + s.  Slots are written upwards and read from at or above
// the slot being written (n >= 1), so one thread can do it in place.
template <typename T, int VEC>
__device__ __forceinline__ void move_conv_state(const T* __restrict__ row0, long long ld, float* __restrict__ st, int n, int p0,
                                                int K, int C, int c) {
    for (int s = 0; s < K; ++s) {
        float v[VEC];
        conv_input<T, VEC>(row0, ld, st, n - K + s, p0, K, C, c, v);
        stv<VEC>(st + (long long)s * C + c, v);
    }
}

// TAPS: compile-time number of taps (inputs slide through registers), or 0 (inputs are read again per tap)
template <typename T, typename TO, int VEC, int TAPS>
__global__ void __launch_bounds__(128)
conv_silu_kernel(const T* __restrict__ proj, long long ld, const float* __restrict__ conv_w, const float* __restrict__ bias,
                 float* __restrict__ conv_state, TO* __restrict__ out, long long ld_out, const int* __restrict__ q_start,
                 const int* __restrict__ n_new, const int* __restrict__ seq_ids, int Tn, int C, int taps, int TT, int move) {
    const int c = (blockIdx.x * 128 + threadIdx.x) * VEC;
    if (c >= C) return;
    const int b = blockIdx.z, t0 = blockIdx.y * TT, t1 = min(t0 + TT, Tn);
    const int n = n_new != nullptr ? min(n_new[b], Tn) : Tn;
    const int line = seq_ids != nullptr ? seq_ids[b] : b;
    const int p0 = q_start[b];
    const int K = (TAPS > 0 ? TAPS : taps) - 1;
    float* st = conv_state + (long long)line * K * C;
    const T* row0 = proj + (long long)b * Tn * ld;
    TO* orow = out + (long long)b * Tn * ld_out + c;
    float bv[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) bv[i] = bias != nullptr ? bias[c + i] : 0.f;
    const int te = min(t1, n);
    if (TAPS > 0) {
        constexpr int NT = TAPS > 0 ? TAPS : 1;
        float w[NT][VEC], win[NT][VEC];
#pragma unroll
        for (int j = 0; j < NT; ++j)
#pragma unroll
            for (int i = 0; i < VEC; ++i) w[j][i] = conv_w[(long long)j * C + c + i];
        if (t0 < te) {
#pragma unroll
            for (int j = 0; j + 1 < NT; ++j) conv_input<T, VEC>(row0, ld, st, t0 - (NT - 1) + j, p0, K, C, c, win[j + 1]);
        }
#pragma unroll 4
        for (int t = t0; t < te; ++t) {
            float acc[VEC];
#pragma unroll
            for (int j = 0; j + 1 < NT; ++j)
#pragma unroll
                for (int i = 0; i < VEC; ++i) win[j][i] = win[j + 1][i];
            ldv<VEC>(row0 + (long long)t * ld + c, win[NT - 1]);
#pragma unroll
            for (int i = 0; i < VEC; ++i) {
                acc[i] = bv[i];
#pragma unroll
                for (int j = 0; j < NT; ++j) acc[i] = fmaf(w[j][i], win[j][i], acc[i]);
                acc[i] = ScanMath<TO>::silu(acc[i]);
            }
            stv<VEC>(orow + (long long)t * ld_out, acc);
        }
    } else {
        for (int t = t0; t < te; ++t) {
            float acc[VEC], v[VEC];
#pragma unroll
            for (int i = 0; i < VEC; ++i) acc[i] = bv[i];
            for (int j = 0; j <= K; ++j) {
                conv_input<T, VEC>(row0, ld, st, t - K + j, p0, K, C, c, v);
#pragma unroll
                for (int i = 0; i < VEC; ++i) acc[i] = fmaf(conv_w[(long long)j * C + c + i], v[i], acc[i]);
            }
#pragma unroll
            for (int i = 0; i < VEC; ++i) acc[i] = ScanMath<TO>::silu(acc[i]);
            stv<VEC>(orow + (long long)t * ld_out, acc);
        }
    }
    float zero[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) zero[i] = 0.f;
    for (int t = max(t0, n); t < t1; ++t) stv<VEC>(orow + (long long)t * ld_out, zero);
    if (move && n > 0) move_conv_state<T, VEC>(row0, ld, st, n, p0, K, C, c);
}

// Long 16-bit steps: a thread convolves STRIP tokens of eight channels, all of whose STRIP + TAPS - 1 rows it asks for at once
// (the overlap between strips is served by the caches).  Does not move the state.
constexpr int STRIP = 8;

template <int TAPS>
__global__ void __launch_bounds__(128)
conv_silu_strip_kernel(const bf16* __restrict__ proj, long long ld, const float* __restrict__ conv_w,
                       const float* __restrict__ bias, const float* __restrict__ conv_state, bf16* __restrict__ out,
                       long long ld_out, const int* __restrict__ q_start, const int* __restrict__ n_new,
                       const int* __restrict__ seq_ids, int Tn, int C) {
    constexpr int K = TAPS - 1;
    const int c = (blockIdx.x * 128 + threadIdx.x) * 8;
    if (c >= C) return;
    const int b = blockIdx.z, t0 = blockIdx.y * STRIP;
    const int n = n_new != nullptr ? min(n_new[b], Tn) : Tn;
    const bf16* row0 = proj + (long long)b * Tn * ld + c;
    bf16* orow = out + (long long)b * Tn * ld_out + c;
    bf16x8 raw[STRIP + K];
#pragma unroll
    for (int j = 0; j < STRIP + K; ++j) {
        const int t = t0 - K + j;
        if (t >= 0 && t < n) raw[j] = *reinterpret_cast<const bf16x8*>(row0 + (long long)t * ld);
    }
    float bv[8], w[TAPS][8];
#pragma unroll
    for (int i = 0; i < 8; ++i) bv[i] = 0.f;
    if (bias != nullptr) ldv<8>(bias + c, bv);
#pragma unroll
    for (int j = 0; j < TAPS; ++j) ldv<8>(conv_w + (long long)j * C + c, w[j]);
    float win[TAPS][8];
    const int line = seq_ids != nullptr ? seq_ids[b] : b;
#pragma unroll
    for (int j = 0; j < K; ++j) {
        if (t0 - K + j >= 0) {
            unpack8(raw[j], win[j + 1]);
        } else {                                               // ahead of the step: the line's state, zeros ahead of the sequence
            conv_input<bf16, 8>(nullptr, 0, conv_state + (long long)line * K * C, t0 - K + j, q_start[b], K, C, c, win[j + 1]);
        }
    }
#pragma unroll
    for (int g = 0; g < STRIP; ++g) {
        const int t = t0 + g;
        if (t >= Tn) break;
        float acc[8];
#pragma unroll
        for (int j = 0; j < K; ++j)
#pragma unroll
            for (int i = 0; i < 8; ++i) win[j][i] = win[j + 1][i];
        if (t < n) {
            unpack8(raw[g + K], win[K]);
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                acc[i] = bv[i];
#pragma unroll
                for (int j = 0; j < TAPS; ++j) acc[i] = fmaf(w[j][i], win[j][i], acc[i]);
                acc[i] = ScanMath<bf16>::silu(acc[i]);
            }
        } else {
#pragma unroll
            for (int i = 0; i < 8; ++i) acc[i] = 0.f;
        }
        stv<8>(orow + (long long)t * ld_out, acc);
    }
}

template <typename T>
__global__ void conv_state_kernel(const T* __restrict__ proj, long long ld, float* __restrict__ conv_state,
                                  const int* __restrict__ q_start, const int* __restrict__ n_new,
                                  const int* __restrict__ seq_ids, int Tn, int C, int taps) {
    const int c = blockIdx.x * blockDim.x + threadIdx.x, b = blockIdx.y;
    if (c >= C) return;
    const int n = n_new != nullptr ? min(n_new[b], Tn) : Tn;
    if (n <= 0) return;
    const int line = seq_ids != nullptr ? seq_ids[b] : b;
    move_conv_state<T, 1>(proj + (long long)b * Tn * ld, ld, conv_state + (long long)line * (taps - 1) * C, n, q_start[b],
                          taps - 1, C, c);
}

// ---- selective scan --------------------------------------------------------------------------------------------------------
// v[j] of lane r (r = its place among R neighbouring lanes) -> the sum over the R lanes of v[r], R - 1 shuffles in all
template <int R>
__device__ __forceinline__ float transpose_sum(float (&v)[R], int r) {
#pragma unroll
    for (int o = 1; o < R; o <<= 1) {
        const bool up = (r & o) != 0;
#pragma unroll
        for (int j = 0; j < R; j += 2 * o) {
            const float keep = up ? v[j + o] : v[j], give = up ? v[j] : v[j + o];
            v[j] = keep + __shfl_xor_sync(0xffffffffu, give, o);
        }
    }
    return v[0];
}

// Half of the CTA scans block i while the other half prepares block i + 1 (step sizes), finishes block i - 1 (skip term, gate,
// store) and fetches block i + 2: one barrier per block of TS tokens.
constexpr int SS_SCAN = 128, SS_HELP = 128, SS_BUFS = 4;

// NS states of each of CPT neighbouring channels per scanning thread, R neighbouring lanes share them
template <typename T, int NS, int R, int CPT, int TS>
struct ScanSmem {
    static constexpr int CH = SS_SCAN / R * CPT, NP = NS * R;
    struct Buf {
        float B[TS][NP], Cm[TS][NP];
        float dt[TS][CH];                                  // pre-activations, then step sizes
        float u[TS][CH];                                   // dt * x, then sum_n S C
        T x[TS][CH], z[TS][CH];
    } buf[SS_BUFS];
};

template <typename T, int NS, int R, int CPT, int TS>
__global__ void __launch_bounds__(SS_SCAN + SS_HELP)
selective_scan_kernel(const T* __restrict__ x, long long ld_x, const float* __restrict__ dt, long long ld_dt,
                      const float* __restrict__ dt_bias, const float* __restrict__ bc, long long ld_bc, int b_off, int c_off,
                      const T* __restrict__ z, long long ld_z, const float* __restrict__ a_log, const float* __restrict__ dskip,
                      float* __restrict__ S, T* __restrict__ out, long long ld_out, const int* __restrict__ q_start,
                      const int* __restrict__ n_new, const int* __restrict__ seq_ids, int Tn, int C, int N, int async) {
    using Sm = ScanSmem<T, NS, R, CPT, TS>;
    constexpr int CH = Sm::CH, NP = Sm::NP, THREADS = SS_SCAN + SS_HELP;
    static_assert(TS % R == 0 && NS % 4 == 0, "tokens come in groups of R, states in groups of 4");
    extern __shared__ __align__(16) unsigned char smem_raw[];
    Sm& sm = *reinterpret_cast<Sm*>(smem_raw);
    const int tid = threadIdx.x;
    const bool helper = tid >= SS_SCAN;
    const int c0 = blockIdx.x * CH, b = blockIdx.y;
    const int n = n_new != nullptr ? min(n_new[b], Tn) : Tn;
    const long long row0 = (long long)b * Tn;
    const int nch = min(CH, C - c0);
    for (int idx = tid; idx < (Tn - max(n, 0)) * nch; idx += THREADS)                        // padding rows
        stf(out + (row0 + max(n, 0) + idx / nch) * ld_out + c0 + idx % nch, 0.f);
    if (n <= 0) return;
    const int line = seq_ids != nullptr ? seq_ids[b] : b;
    const bool fresh = q_start[b] == 0;
    const int tiles = (n + TS - 1) / TS;
    // columns N .. NP - 1 of B and C are zeros in all buffers and stay so
    if (N < NP)
        for (int idx = tid; idx < SS_BUFS * TS * (NP - N); idx += THREADS) {
            const int k = idx / (TS * (NP - N)), q = idx % (TS * (NP - N));
            sm.buf[k].B[q / (NP - N)][N + q % (NP - N)] = 0.f;
            sm.buf[k].Cm[q / (NP - N)][N + q % (NP - N)] = 0.f;
        }
    if (!helper) {
        const int r = tid % R, cl = tid / R * CPT;
        float* Sc = S + ((long long)line * C + c0 + cl) * N;
        uint64_t s[CPT][NS / 2], a2[CPT][NS / 2];
#pragma unroll
        for (int m = 0; m < CPT; ++m)
#pragma unroll
            for (int j = 0; j < NS / 2; ++j) {
                float sv[2], av[2];
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int i = r * NS + 2 * j + e;
                    const bool ok = cl + m < nch && i < N;
                    sv[e] = (ok && !fresh) ? Sc[(long long)m * N + i] : 0.f;
                    av[e] = ok ? ScanDecay<T>::rate(-expf(a_log[(long long)(c0 + cl + m) * N + i])) : 0.f;
                }
                s[m][j] = pair2(sv[0], sv[1]);
                a2[m][j] = pair2(av[0], av[1]);
            }
        __syncthreads();
        for (int it = 0; it <= tiles + 1; ++it) {
            if (it >= 1 && it <= tiles) {
                typename Sm::Buf& d = sm.buf[(it - 1) & (SS_BUFS - 1)];
                const int top = (min(TS, n - (it - 1) * TS) + R - 1) / R * R;
                for (int g0 = 0; g0 < top; g0 += R) {
                    float y[CPT][R];
#pragma unroll
                    for (int q = 0; q < R; ++q) {
                        uint64_t dv[CPT], u[CPT], acc[CPT];
#pragma unroll
                        for (int m = 0; m < CPT; ++m) {
                            const float dvs = d.dt[g0 + q][cl + m], us = d.u[g0 + q][cl + m];
                            dv[m] = pair2(dvs, dvs), u[m] = pair2(us, us), acc[m] = 0ull;
                        }
#pragma unroll
                        for (int j = 0; j < NS; j += 4) {
                            const ulonglong2 bv = *reinterpret_cast<const ulonglong2*>(&d.B[g0 + q][r * NS + j]);
                            const ulonglong2 cv = *reinterpret_cast<const ulonglong2*>(&d.Cm[g0 + q][r * NS + j]);
#pragma unroll
                            for (int m = 0; m < CPT; ++m) {
                                const uint64_t g01 = ScanDecay<T>::at2(dv[m], a2[m][j / 2]);
                                const uint64_t g23 = ScanDecay<T>::at2(dv[m], a2[m][j / 2 + 1]);
                                s[m][j / 2] = fma2(g01, s[m][j / 2], mul2(u[m], bv.x));
                                s[m][j / 2 + 1] = fma2(g23, s[m][j / 2 + 1], mul2(u[m], bv.y));
                                acc[m] = fma2(s[m][j / 2], cv.x, acc[m]);
                                acc[m] = fma2(s[m][j / 2 + 1], cv.y, acc[m]);
                            }
                        }
#pragma unroll
                        for (int m = 0; m < CPT; ++m) {
                            float lo, hi;
                            unpair2(acc[m], lo, hi);
                            y[m][q] = lo + hi;
                        }
                    }
                    // every lane of the channel has read its u of these tokens (the shuffles wait for them): y takes their place
#pragma unroll
                    for (int m = 0; m < CPT; ++m) {
                        const float v = transpose_sum<R>(y[m], r);
                        d.u[g0 + r][cl + m] = v;
                    }
                }
            }
            __syncthreads();
        }
#pragma unroll
        for (int m = 0; m < CPT; ++m)
#pragma unroll
            for (int j = 0; j < NS / 2; ++j) {
                float lo, hi;
                unpair2(s[m][j], lo, hi);
                const int i = r * NS + 2 * j;
                if (cl + m < nch && i < N) Sc[(long long)m * N + i] = lo;
                if (cl + m < nch && i + 1 < N) Sc[(long long)m * N + i + 1] = hi;
            }
        return;
    }
    constexpr int XV = 16 / sizeof(T);                       // elements of T per 16 bytes
    constexpr int CX = CH / XV;                              // such pieces per token
    const int ht = tid - SS_SCAN;
    auto fetch = [&](int tile) {
        typename Sm::Buf& d = sm.buf[tile & (SS_BUFS - 1)];
        const int t0 = tile * TS, cnt = min(TS, n - t0);
        if (async) {
            const int n4 = N / 4;
            for (int idx = ht; idx < cnt * n4; idx += SS_HELP) {
                const int tt = idx / n4, i = (idx - tt * n4) * 4;
                const float* src = bc + (row0 + t0 + tt) * ld_bc + i;
                mma::cp_async16((uint32_t)__cvta_generic_to_shared(&d.B[tt][i]), src + b_off, true);
                mma::cp_async16((uint32_t)__cvta_generic_to_shared(&d.Cm[tt][i]), src + c_off, true);
            }
            for (int idx = ht; idx < cnt * (CH / 4); idx += SS_HELP) {
                const int tt = idx / (CH / 4), i = (idx % (CH / 4)) * 4;
                const bool ok = i < nch;
                mma::cp_async16((uint32_t)__cvta_generic_to_shared(&d.dt[tt][i]), dt + (row0 + t0 + tt) * ld_dt + c0 + (ok ? i : 0), ok);
            }
            for (int idx = ht; idx < cnt * CX; idx += SS_HELP) {
                const int tt = idx / CX, i = (idx % CX) * XV;
                const bool ok = i < nch;
                const long long at = row0 + t0 + tt;
                mma::cp_async16((uint32_t)__cvta_generic_to_shared(&d.x[tt][i]), x + at * ld_x + c0 + (ok ? i : 0), ok);
                mma::cp_async16((uint32_t)__cvta_generic_to_shared(&d.z[tt][i]), z + at * ld_z + c0 + (ok ? i : 0), ok);
            }
        } else {
            for (int idx = ht; idx < cnt * N; idx += SS_HELP) {
                const int tt = idx / N, i = idx % N;
                const float* src = bc + (row0 + t0 + tt) * ld_bc + i;
                d.B[tt][i] = src[b_off];
                d.Cm[tt][i] = src[c_off];
            }
            for (int idx = ht; idx < cnt * CH; idx += SS_HELP) {
                const int tt = idx / CH, i = idx % CH;
                const bool ok = i < nch;
                const long long at = row0 + t0 + tt;
                d.dt[tt][i] = ok ? dt[at * ld_dt + c0 + i] : 0.f;
                stf(&d.x[tt][i], ok ? ldf(x + at * ld_x + c0 + i) : 0.f);
                stf(&d.z[tt][i], ok ? ldf(z + at * ld_z + c0 + i) : 0.f);
            }
        }
    };
    // a helper prepares and finishes VP neighbouring channels of every ROWS-th token, always the same channels
    constexpr int VP = 2, PT = CH / VP, ROWS = SS_HELP / PT;
    static_assert(SS_HELP % PT == 0 && CH % VP == 0, "channel slices");
    const int pi = ht % PT * VP, prow = ht / PT;
    float bias[VP], dsk[VP];
#pragma unroll
    for (int v = 0; v < VP; ++v) {
        bias[v] = (dt_bias != nullptr && pi + v < nch) ? dt_bias[c0 + pi + v] : 0.f;
        dsk[v] = pi + v < nch ? dskip[c0 + pi + v] : 0.f;
    }
    fetch(0);
    mma::cp_async_commit();
    __syncthreads();
    for (int it = 0; it <= tiles + 1; ++it) {
        if (it + 1 < tiles) fetch(it + 1);
        mma::cp_async_commit();
        mma::cp_async_wait<1>();
        asm volatile("bar.sync 1, %0;" ::"n"(SS_HELP) : "memory");       // block `it` has arrived for every helper
        if (it < tiles) {
            typename Sm::Buf& d = sm.buf[it & (SS_BUFS - 1)];
            const int cnt = min(TS, n - it * TS), top = (cnt + R - 1) / R * R;
            for (int tt = prow; tt < top; tt += ROWS) {                  // step sizes; tokens past the end: no step
#pragma unroll
                for (int v = 0; v < VP; ++v) {
                    const bool ok = tt < cnt && pi + v < nch;
                    const float step = ok ? ScanMath<T>::softplus(d.dt[tt][pi + v] + bias[v]) : 0.f;
                    d.dt[tt][pi + v] = step;
                    d.u[tt][pi + v] = ok ? step * ldf(&d.x[tt][pi + v]) : 0.f;
                }
            }
            for (int idx = ht; idx < (top - cnt) * N; idx += SS_HELP) {  // rows that no copy has filled
                d.B[cnt + idx / N][idx % N] = 0.f;
                d.Cm[cnt + idx / N][idx % N] = 0.f;
            }
        }
        if (it >= 2) {
            typename Sm::Buf& d = sm.buf[(it - 2) & (SS_BUFS - 1)];
            const int t0 = (it - 2) * TS, cnt = min(TS, n - t0);
            for (int tt = prow; tt < cnt; tt += ROWS) {
                float v[VP];
#pragma unroll
                for (int w = 0; w < VP; ++w)
                    v[w] = fmaf(dsk[w], ldf(&d.x[tt][pi + w]), d.u[tt][pi + w]) * ScanMath<T>::silu(ldf(&d.z[tt][pi + w]));
                T* dst = out + (row0 + t0 + tt) * ld_out + c0 + pi;
                if (async && pi + 1 < nch) {
                    if (sizeof(T) == 4) *reinterpret_cast<float2*>(dst) = make_float2(v[0], v[1]);
                    else *reinterpret_cast<uint32_t*>(dst) = mma::pack2(v[0], v[1]);
                } else {
#pragma unroll
                    for (int w = 0; w < VP; ++w)
                        if (pi + w < nch) stf(dst + w, v[w]);
                }
            }
        }
        __syncthreads();
    }
}

template <typename T, int NS, int R, int CPT, int TS>
int launch_selective(const void* x, long long ld_x, const float* dt, long long ld_dt, const float* dt_bias, const float* bc,
                     long long ld_bc, int b_off, int c_off, const void* z, long long ld_z, const float* a_log,
                     const float* dskip, float* S, void* out, long long ld_out, const int* q_start, const int* n_new,
                     const int* seq_ids, int B, int Tn, int C, int N, cudaStream_t st) {
    using Sm = ScanSmem<T, NS, R, CPT, TS>;
    constexpr size_t smem = sizeof(Sm);
    auto al = [](const void* p) { return ((uintptr_t)p % 16) == 0; };
    constexpr int XV = 16 / sizeof(T);
    const int async = Sm::CH % XV == 0 && C % XV == 0 && ld_x % XV == 0 && ld_z % XV == 0 && ld_out % XV == 0 && ld_dt % 4 == 0 &&
                      ld_bc % 4 == 0 && b_off % 4 == 0 && c_off % 4 == 0 && N % 4 == 0 && al(x) && al(z) && al(dt) && al(bc) && al(out);
    auto kern = selective_scan_kernel<T, NS, R, CPT, TS>;
    if (smem > 48 * 1024) NXD_CHECK_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    dim3 grid((C + Sm::CH - 1) / Sm::CH, B);
    kern<<<grid, SS_SCAN + SS_HELP, smem, st>>>((const T*)x, ld_x, dt, ld_dt, dt_bias, bc, ld_bc, b_off, c_off, (const T*)z, ld_z, a_log,
                                         dskip, S, (T*)out, ld_out, q_start, n_new, seq_ids, Tn, C, N, async);
    NXD_LAUNCH_CHECK();
    return 0;
}

// One token per row.  A CTA takes 32 channels (four lanes each) of STEP_ROWS rows, so that the low-rank weights that make the step
// sizes, dt_c = softplus(<dt_w[c], p[row]> + bias_c), are read once for those rows; every state is read and written once.
constexpr int STEP_ROWS = 4, STEP_THREADS = 128;

template <typename T, bool VEC>
__global__ void __launch_bounds__(STEP_THREADS)
selective_step_kernel(const T* __restrict__ x, long long ld_x, const T* __restrict__ dt_w, int rank,
                      const float* __restrict__ dt_bias, const float* __restrict__ p, long long ld_p, int b_off, int c_off,
                      const T* __restrict__ z, long long ld_z, const float* __restrict__ a_log, const float* __restrict__ dskip,
                      float* __restrict__ S, T* __restrict__ out, long long ld_out, const int* __restrict__ q_start,
                      const int* __restrict__ seq_ids, int B, int C, int N) {
    extern __shared__ __align__(16) float smem[];              // [STEP_ROWS][rank + 2 N, padded to 4]
    const int pitch = (rank + 2 * N + 3) & ~3;
    const int tid = threadIdx.x, r = tid & 3, c = blockIdx.x * 32 + (tid >> 2);
    const int b0 = blockIdx.y * STEP_ROWS, nb = min(STEP_ROWS, B - b0);
    const bool ok = c < C;
    // up to 16 states (one 16-byte piece per lane): they and their decay rates are on their way before anything else
    const bool small = VEC && N <= 16, mine = small && ok && r * 4 < N;
    float pre[STEP_ROWS][4], rate[4];
    if (mine) {
        ldv<4>(a_log + (long long)c * N + r * 4, rate);
#pragma unroll
        for (int q = 0; q < STEP_ROWS; ++q)
            if (q < nb) ldv<4>(S + ((long long)(seq_ids != nullptr ? seq_ids[b0 + q] : b0 + q) * C + c) * N + r * 4, pre[q]);
#pragma unroll
        for (int e = 0; e < 4; ++e) rate[e] = ScanDecay<T>::rate(-expf(rate[e]));
    }
    const T* wr = dt_w + (long long)(ok ? c : 0) * rank;       // rank is a multiple of 8
    constexpr int AHEAD = 4;                                   // pieces of the weights that are asked for up front
    float w[AHEAD][8];
#pragma unroll
    for (int j = 0; j < AHEAD; ++j)
        if (r * 8 + 32 * j < rank) ldv<8>(wr + r * 8 + 32 * j, w[j]);
    if (VEC && ((ld_p | b_off | c_off) & 3) == 0 && ((uintptr_t)p & 15) == 0) {
        const int p4 = pitch / 4, r4 = rank / 4, n4 = N / 4;
        for (int q = tid >> 5; q < nb; q += STEP_THREADS / 32) {          // a warp per row
            const float* row = p + (long long)(b0 + q) * ld_p;
#pragma unroll 4
            for (int i = tid & 31; i < p4; i += 32) {
                const int at = i < r4 ? 4 * i : (i < r4 + n4 ? b_off + 4 * (i - r4) : c_off + 4 * (i - r4 - n4));
                *reinterpret_cast<float4*>(smem + q * pitch + 4 * i) = *reinterpret_cast<const float4*>(row + at);
            }
        }
    } else {
        for (int idx = tid; idx < nb * pitch; idx += STEP_THREADS) {
            const int q = idx / pitch, i = idx - q * pitch;
            const float* row = p + (long long)(b0 + q) * ld_p;
            smem[idx] = i < rank ? row[i] : (i < rank + N ? row[b_off + i - rank] : (i < rank + 2 * N ? row[c_off + i - rank - N] : 0.f));
        }
    }
    __syncthreads();
    float acc[STEP_ROWS];
#pragma unroll
    for (int q = 0; q < STEP_ROWS; ++q) acc[q] = 0.f;
    auto products = [&](int k, const float* v8) {
#pragma unroll
        for (int q = 0; q < STEP_ROWS; ++q)
            if (q < nb) {
                const float4 u = *reinterpret_cast<const float4*>(smem + q * pitch + k);
                const float4 v = *reinterpret_cast<const float4*>(smem + q * pitch + k + 4);
                acc[q] += fmaf(v8[0], u.x, fmaf(v8[1], u.y, fmaf(v8[2], u.z, v8[3] * u.w))) +
                          fmaf(v8[4], v.x, fmaf(v8[5], v.y, fmaf(v8[6], v.z, v8[7] * v.w)));
            }
    };
#pragma unroll
    for (int j = 0; j < AHEAD; ++j)
        if (r * 8 + 32 * j < rank) products(r * 8 + 32 * j, w[j]);
#pragma unroll 4
    for (int k = r * 8 + 32 * AHEAD; k < rank; k += 32) {
        float v8[8];
        ldv<8>(wr + k, v8);
        products(k, v8);
    }
    // lane r of a channel takes row r: its sum, its step size, in the end its output
    const float sum = transpose_sum<STEP_ROWS>(acc, r);
    const int br = b0 + r;
    const bool mine_row = ok && r < nb;
    float step_r = 0.f, x_r = 0.f;
    if (mine_row) {
        step_r = ScanMath<T>::softplus(sum + (dt_bias != nullptr ? dt_bias[c] : 0.f));
        x_r = ldf(x + (long long)br * ld_x + c);
    }
    float y[STEP_ROWS];
#pragma unroll
    for (int q = 0; q < STEP_ROWS; ++q) {
        const int src = (tid & 31 & ~3) | q;
        const float step = __shfl_sync(0xffffffffu, step_r, src), u = step * __shfl_sync(0xffffffffu, x_r, src);
        y[q] = 0.f;
        if (!ok || q >= nb) continue;
        const int b = b0 + q, line = seq_ids != nullptr ? seq_ids[b] : b;
        const bool fresh = q_start[b] == 0;
        const float* Bs = smem + q * pitch + rank;
        const float* Cs = Bs + N;
        float* Sc = S + ((long long)line * C + c) * N;
        if (mine) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                pre[q][e] = fmaf(ScanDecay<T>::at(step, rate[e]), fresh ? 0.f : pre[q][e], u * Bs[r * 4 + e]);
                y[q] = fmaf(pre[q][e], Cs[r * 4 + e], y[q]);
            }
            stv<4>(Sc + r * 4, pre[q]);
        }
        if (small) continue;
        constexpr int W = VEC ? 4 : 1;
        const float* al = a_log + (long long)c * N;
        for (int i = r * W; i < N; i += 4 * W) {
            float s[W], a[W];
            if (fresh) {
#pragma unroll
                for (int e = 0; e < W; ++e) s[e] = 0.f;
            } else {
                ldv<W>(Sc + i, s);
            }
            ldv<W>(al + i, a);
#pragma unroll
            for (int e = 0; e < W; ++e) {
                s[e] = fmaf(ScanDecay<T>::at(step, ScanDecay<T>::rate(-expf(a[e]))), s[e], u * Bs[i + e]);
                y[q] = fmaf(s[e], Cs[i + e], y[q]);
            }
            stv<W>(Sc + i, s);
        }
    }
    const float yr = transpose_sum<STEP_ROWS>(y, r);
    if (mine_row)
        stf(out + (long long)br * ld_out + c, fmaf(dskip[c], x_r, yr) * ScanMath<T>::silu(ldf(z + (long long)br * ld_z + c)));
}

// ---- state-space heads: one token ------------------------------------------------------------------------------------------
// blockIdx.x: slice of 32 columns, y: head, z: row.  A thread owns VEC neighbouring columns and every ROWS-th state row.  With
// dt == NULL the CTA makes its head's step size itself, <dt_w[h], hin[row]> over the layer's W inputs.
template <typename T, typename TY, int VEC>
__global__ void __launch_bounds__(128)
ssd_step_kernel(const T* __restrict__ xbc, long long ld, int x_off, int b_off, int c_off, const float* __restrict__ dt,
                long long ld_dt, const float* __restrict__ dt_bias, const float* __restrict__ a_log,
                const float* __restrict__ dskip, float* __restrict__ S, TY* __restrict__ y, const int* __restrict__ q_start,
                const int* __restrict__ seq_ids, int H, int G, int N, int P, const T* __restrict__ hin,
                const T* __restrict__ dt_w, int W) {
    constexpr int LC = 32 / VEC, ROWS = 128 / LC;              // lanes per row, rows in flight
    extern __shared__ float smem[];
    float* Bs = smem;                                          // [N]
    float* Cs = Bs + N;                                        // [N]
    __shared__ float red[ROWS][32];
    const int tid = threadIdx.x, lc = tid % LC, rg = tid / LC;
    const int p0 = blockIdx.x * 32 + lc * VEC, h = blockIdx.y, b = blockIdx.z, g = h / (H / G);
    const T* row = xbc + (long long)b * ld;
    for (int i = tid; i < N; i += 128) {
        Bs[i] = ldf(row + b_off + g * N + i);
        Cs[i] = ldf(row + c_off + g * N + i);
    }
    float pre = 0.f;
    if (dt != nullptr) {
        pre = dt[(long long)b * ld_dt + h];
    } else {
        const T* hr = hin + (long long)b * W;
        const T* wr = dt_w + (long long)h * W;
        if (W % 8 == 0) {
#pragma unroll 2
            for (int c = tid * 8; c < W; c += 128 * 8) {
                float u8[8], w8[8];
                ldv<8>(hr + c, u8);
                ldv<8>(wr + c, w8);
#pragma unroll
                for (int i = 0; i < 8; ++i) pre = fmaf(u8[i], w8[i], pre);
            }
        } else {
            for (int c = tid; c < W; c += 128) pre = fmaf(ldf(hr + c), ldf(wr + c), pre);
        }
        pre = block_sum(pre, &red[0][0]);
        __syncthreads();                                       // red is used again below
    }
    const float step = softplus_f(pre + (dt_bias != nullptr ? dt_bias[h] : 0.f));
    const float decay = decay_exp(-expf(a_log[h]) * step);
    const bool fresh = q_start[b] == 0, ok = p0 < P;
    const int line = seq_ids != nullptr ? seq_ids[b] : b;
    float xv[VEC], u[VEC], acc[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
        xv[i] = ok ? ldf(row + x_off + (long long)h * P + p0 + i) : 0.f;
        u[i] = step * xv[i];
        acc[i] = 0.f;
    }
    __syncthreads();
    float* Sg = S + ((long long)line * H + h) * N * P + p0;
    if (ok) {
#pragma unroll 4
        for (int i = rg; i < N; i += ROWS) {
            float v[VEC];
            if (fresh) {
#pragma unroll
                for (int q = 0; q < VEC; ++q) v[q] = 0.f;
            } else {
                ldv<VEC>(Sg + (long long)i * P, v);
            }
            const float bv = Bs[i], cv = Cs[i];
#pragma unroll
            for (int q = 0; q < VEC; ++q) {
                v[q] = fmaf(decay, v[q], u[q] * bv);
                acc[q] = fmaf(v[q], cv, acc[q]);
            }
            stv<VEC>(Sg + (long long)i * P, v);
        }
    }
#pragma unroll
    for (int q = 0; q < VEC; ++q) red[rg][lc * VEC + q] = acc[q];
    __syncthreads();
    if (tid < 32) {
        const int p = blockIdx.x * 32 + tid;
        if (p < P) {
            float o = 0.f;
#pragma unroll
            for (int q = 0; q < ROWS; ++q) o += red[q][tid];
            const float xp = ldf(row + x_off + (long long)h * P + p);
            stf(y + ((long long)b * H + h) * P + p, fmaf(dskip[h], xp, o));
        }
    }
}

// ---- state-space heads: token by token -------------------------------------------------------------------------------------
// A thread keeps NPT rows of one state column in registers; the R lanes that share a column sit cpw = 32 / R lanes apart.
// Slices are padded to NPT + 4 floats in shared memory, so that the R 16-byte reads of a warp fall into different banks.
template <typename T, typename TY, int NPT>
__global__ void __launch_bounds__(128)
ssd_scan_kernel(const T* __restrict__ xbc, long long ld, int x_off, int b_off, int c_off, const float* __restrict__ dt,
                long long ld_dt, const float* __restrict__ dt_bias, const float* __restrict__ a_log,
                const float* __restrict__ dskip, float* __restrict__ S, TY* __restrict__ y, const int* __restrict__ q_start,
                const int* __restrict__ n_new, const int* __restrict__ seq_ids, int Tn, int H, int G, int N, int P, int R) {
    constexpr int PITCH = NPT + 4, TS = 16;
    extern __shared__ __align__(16) float smem[];
    const int DS = R * PITCH, CT = 128 / R, cpw = 32 / R, NP = R * NPT;
    float* Bs = smem;                        // [TS][DS]
    float* Cs = Bs + TS * DS;                // [TS][DS]
    float* xs = Cs + TS * DS;                // [TS][CT]
    __shared__ float sd[TS], sg[TS];         // step, decay
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, r = lane / cpw, cl = warp * cpw + lane % cpw;
    const int col0 = blockIdx.x * CT, col = col0 + cl, h = blockIdx.y, b = blockIdx.z, g = h / (H / G);
    const int n = n_new != nullptr ? min(n_new[b], Tn) : Tn;
    const long long row0 = (long long)b * Tn;
    if (r == 0 && col < P)
        for (int t = max(n, 0); t < Tn; ++t) stf(y + ((row0 + t) * H + h) * P + col, 0.f);
    if (n <= 0) return;
    const int line = seq_ids != nullptr ? seq_ids[b] : b;
    float* Sg = S + ((long long)line * H + h) * N * P + col;
    const bool fresh = q_start[b] == 0;
    float s[NPT];
#pragma unroll
    for (int j = 0; j < NPT; ++j) {
        const int i = r * NPT + j;
        s[j] = (!fresh && i < N && col < P) ? Sg[(long long)i * P] : 0.f;
    }
    const float a = expf(a_log[h]), dsk = dskip[h];
    for (int t0 = 0; t0 < n; t0 += TS) {
        const int cnt = min(TS, n - t0);
        __syncthreads();
        for (int idx = tid; idx < cnt * NP; idx += 128) {
            const int tt = idx / NP, i = idx - tt * NP;
            const T* row = xbc + (row0 + t0 + tt) * ld;
            const int at = tt * DS + (i / NPT) * PITCH + (i % NPT);
            Bs[at] = i < N ? ldf(row + b_off + g * N + i) : 0.f;
            Cs[at] = i < N ? ldf(row + c_off + g * N + i) : 0.f;
        }
        for (int idx = tid; idx < cnt * CT; idx += 128) {
            const int tt = idx / CT, i = idx - tt * CT;
            xs[idx] = col0 + i < P ? ldf(xbc + (row0 + t0 + tt) * ld + x_off + (long long)h * P + col0 + i) : 0.f;
        }
        if (tid < cnt) {
            const float step = softplus_f(dt[(row0 + t0 + tid) * ld_dt + h] + (dt_bias != nullptr ? dt_bias[h] : 0.f));
            sd[tid] = step;
            sg[tid] = decay_exp(-a * step);
        }
        __syncthreads();
        for (int tt = 0; tt < cnt; ++tt) {
            const float xv = xs[tt * CT + cl], u = sd[tt] * xv, dec = sg[tt];
            const float4* b4 = reinterpret_cast<const float4*>(Bs + tt * DS + r * PITCH);
            const float4* c4 = reinterpret_cast<const float4*>(Cs + tt * DS + r * PITCH);
            float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int v = 0; v < NPT / 4; ++v) {
                const float4 bv = b4[v], cv = c4[v];
                s[4 * v] = fmaf(dec, s[4 * v], u * bv.x), s[4 * v + 1] = fmaf(dec, s[4 * v + 1], u * bv.y);
                s[4 * v + 2] = fmaf(dec, s[4 * v + 2], u * bv.z), s[4 * v + 3] = fmaf(dec, s[4 * v + 3], u * bv.w);
                acc[0] = fmaf(s[4 * v], cv.x, acc[0]), acc[1] = fmaf(s[4 * v + 1], cv.y, acc[1]);
                acc[2] = fmaf(s[4 * v + 2], cv.z, acc[2]), acc[3] = fmaf(s[4 * v + 3], cv.w, acc[3]);
            }
            float o = (acc[0] + acc[1]) + (acc[2] + acc[3]);
            for (int off = cpw; off < 32; off <<= 1) o += __shfl_xor_sync(0xffffffffu, o, off);
            if (r == 0 && col < P) stf(y + ((row0 + t0 + tt) * H + h) * P + col, fmaf(dsk, xv, o));
        }
    }
    if (col < P) {
#pragma unroll
        for (int j = 0; j < NPT; ++j) {
            const int i = r * NPT + j;
            if (i < N) Sg[(long long)i * P] = s[j];
        }
    }
}

// ---- state-space heads: chunks of 64 tokens on the tensor cores --------------------------------------------------------------
// One CTA: PT = 16 * WARPS columns of one head of one row, all chunks in order.  With cum_t the running sum of the chunk's log
// decays,
//     y_t = exp(cum_t) S_0^T C_t + sum_{s <= t} (C_t . B_s) exp(cum_t - cum_s) dt_s x_s  (+ D x_t)
//     S_L = exp(cum_L) S_0 + sum_s exp(cum_L - cum_s) dt_s B_s x_s^T
// Every exponent is a sum of log decays and never positive.  A warp owns 16 columns: their state (transposed, [16, NPAD]) sits in
// accumulator registers, whose layout is the B operand of S_0^T C and the accumulator of the update at once.  The score
// tile is computed once per CTA (a warp: 64 / WARPS rows) and passed through shared memory.
constexpr int CL = 64;                       // tokens per chunk

__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
    const bf162 h = __floats2bfloat162_rn(a, b);
    const float2 f = __bfloat1622float2(h);
    const bf162 l = __floats2bfloat162_rn(a - f.x, b - f.y);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ float2 unpack2(uint32_t v) { return __bfloat1622float2(*reinterpret_cast<const bf162*>(&v)); }

template <int NT, int WARPS>
struct ChunkSmem {
    static constexpr int NPAD = 16 * NT, LDN = NPAD + 8, PT = 16 * WARPS, LDP = PT + 8, LDS = CL + 8;
    bf16 C[2][CL][LDN], B[2][CL][LDN], X[2][CL][LDP];
    bf16 Ph[CL][LDS], Pl[CL][LDS];
    float dt[CL], cum[CL];
};

template <typename TY, int NT, int WARPS>
__global__ void __launch_bounds__(WARPS * 32)
ssd_chunk_kernel(const bf16* __restrict__ xbc, long long ld, int x_off, int b_off, int c_off, const float* __restrict__ dt,
                 long long ld_dt, const float* __restrict__ dt_bias, const float* __restrict__ a_log,
                 const float* __restrict__ dskip, float* __restrict__ S, TY* __restrict__ y, const int* __restrict__ q_start,
                 const int* __restrict__ n_new, const int* __restrict__ seq_ids, int Tn, int H, int G, int N, int P) {
    using Sm = ChunkSmem<NT, WARPS>;
    constexpr int THREADS = WARPS * 32, MT = 4 / WARPS;          // 16-row tiles of the score tile per warp
    extern __shared__ __align__(16) unsigned char smem_raw[];
    Sm& sm = *reinterpret_cast<Sm*>(smem_raw);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, qr = lane >> 2, qc = (lane & 3) * 2;
    const int p_cta = blockIdx.x * Sm::PT, h = blockIdx.y, b = blockIdx.z, g = h / (H / G);
    const int n = n_new != nullptr ? min(n_new[b], Tn) : Tn;
    const long long row0 = (long long)b * Tn;
    const int pw = p_cta + warp * 16;                            // first column of this warp
    {
        const int np = min(Sm::PT, P - p_cta), from = max(n, 0);
        for (int idx = tid; idx < (Tn - from) * np; idx += THREADS)
            stf(y + ((row0 + from + idx / np) * H + h) * P + p_cta + idx % np, 0.f);
    }
    if (n <= 0) return;
    const int line = seq_ids != nullptr ? seq_ids[b] : b;
    float* Sg = S + ((long long)line * H + h) * N * P;
    const bool fresh = q_start[b] == 0;
    const float a = expf(a_log[h]), dsk = dskip[h], dtb = dt_bias != nullptr ? dt_bias[h] : 0.f;

    // state, transposed: tile j holds columns (of N) 8 j .. 8 j + 7; [0], [1]: row pw + qr, [2], [3]: row pw + qr + 8
    float s[2 * NT][4];
#pragma unroll
    for (int j = 0; j < 2 * NT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = j * 8 + qc + (e & 1), p = pw + qr + (e >> 1) * 8;
            s[j][e] = (!fresh && i < N && p < P) ? Sg[(long long)i * P + p] : 0.f;
        }

    auto fetch = [&](int t0, int k) {
        constexpr int CN = Sm::NPAD / 8, CP = Sm::PT / 8;
        for (int idx = tid; idx < CL * CN; idx += THREADS) {
            const int t = idx / CN, i = (idx % CN) * 8;
            const bool ok = t0 + t < n && i < N;
            const bf16* src = xbc + (row0 + (ok ? t0 + t : 0)) * ld + (long long)g * N + (ok ? i : 0);
            mma::cp_async16((uint32_t)__cvta_generic_to_shared(&sm.C[k][t][i]), src + c_off, ok);
            mma::cp_async16((uint32_t)__cvta_generic_to_shared(&sm.B[k][t][i]), src + b_off, ok);
        }
        for (int idx = tid; idx < CL * CP; idx += THREADS) {
            const int t = idx / CP, i = (idx % CP) * 8;
            const bool ok = t0 + t < n && p_cta + i < P;
            const bf16* src = xbc + (row0 + (ok ? t0 + t : 0)) * ld + x_off + (long long)h * P + (ok ? p_cta + i : 0);
            mma::cp_async16((uint32_t)__cvta_generic_to_shared(&sm.X[k][t][i]), src, ok);
        }
        mma::cp_async_commit();
    };
    // raw step sizes of the next chunk, two tokens per lane of warp 0
    float raw0 = 0.f, raw1 = 0.f;
    auto fetch_dt = [&](int t0) {
        if (warp == 0) {
            raw0 = t0 + 2 * lane < n ? dt[(row0 + t0 + 2 * lane) * ld_dt + h] : 0.f;
            raw1 = t0 + 2 * lane + 1 < n ? dt[(row0 + t0 + 2 * lane + 1) * ld_dt + h] : 0.f;
        }
    };
    fetch_dt(0);
    fetch(0, 0);
    int k = 0;
    for (int t0 = 0; t0 < n; t0 += CL, k ^= 1) {
        if (warp == 0) {
            const float d0 = t0 + 2 * lane < n ? softplus_f(raw0 + dtb) : 0.f;
            const float d1 = t0 + 2 * lane + 1 < n ? softplus_f(raw1 + dtb) : 0.f;
            const float l0 = -a * d0, l1 = -a * d1;
            float run = l0 + l1;                                  // inclusive sum over the lanes' pairs
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float up = __shfl_up_sync(0xffffffffu, run, o);
                if (lane >= o) run += up;
            }
            sm.dt[2 * lane] = d0, sm.dt[2 * lane + 1] = d1;
            sm.cum[2 * lane] = run - l1, sm.cum[2 * lane + 1] = run;
        }
        if (t0 + CL < n) {
            fetch(t0 + CL, k ^ 1);
            fetch_dt(t0 + CL);
            mma::cp_async_wait<1>();
        } else {
            mma::cp_async_wait<0>();
        }
        __syncthreads();
        const uint32_t c_addr = (uint32_t)__cvta_generic_to_shared(&sm.C[k][0][0]);
        const uint32_t b_addr = (uint32_t)__cvta_generic_to_shared(&sm.B[k][0][0]);
        const uint32_t x_addr = (uint32_t)__cvta_generic_to_shared(&sm.X[k][0][0]);
        const uint32_t ph_addr = (uint32_t)__cvta_generic_to_shared(&sm.Ph[0][0]);
        const uint32_t pl_addr = (uint32_t)__cvta_generic_to_shared(&sm.Pl[0][0]);

        // decayed scores of this warp's rows, columns up to the diagonal
#pragma unroll
        for (int mi = 0; mi < MT; ++mi) {
            const int m = warp + mi * WARPS;                      // 16-row tile
            float acc[8][4];
#pragma unroll
            for (int j = 0; j < 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
#pragma unroll
            for (int kk = 0; kk < NT; ++kk) {
                uint32_t af[4];
                mma::ldsm_x4(af, c_addr + ((m * 16 + (lane & 15)) * Sm::LDN + kk * 16 + (lane >> 4) * 8) * 2);
#pragma unroll
                for (int np = 0; np < 4; ++np) {
                    if (np <= m) {
                        uint32_t bf[4];
                        mma::ldsm_x4(bf, b_addr + ((np * 16 + (lane & 7) + (lane >> 4) * 8) * Sm::LDN + kk * 16 +
                                                   ((lane >> 3) & 1) * 8) * 2);
                        mma::mma16816(acc[2 * np], af, bf[0], bf[1]);
                        mma::mma16816(acc[2 * np + 1], af, bf[2], bf[3]);
                    }
                }
            }
            const int ta = m * 16 + qr, tb = ta + 8;
            const float ca = sm.cum[ta], cb = sm.cum[tb];
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                if (j <= 2 * m + 1) {
                    const int c0 = j * 8 + qc;
                    const float k0 = sm.cum[c0], k1 = sm.cum[c0 + 1], d0 = sm.dt[c0], d1 = sm.dt[c0 + 1];
                    const float v0 = c0 <= ta ? acc[j][0] * (expf(ca - k0) * d0) : 0.f;
                    const float v1 = c0 + 1 <= ta ? acc[j][1] * (expf(ca - k1) * d1) : 0.f;
                    const float v2 = c0 <= tb ? acc[j][2] * (expf(cb - k0) * d0) : 0.f;
                    const float v3 = c0 + 1 <= tb ? acc[j][3] * (expf(cb - k1) * d1) : 0.f;
                    uint32_t hi, lo;
                    split2(v0, v1, hi, lo);
                    *reinterpret_cast<uint32_t*>(&sm.Ph[ta][c0]) = hi;
                    *reinterpret_cast<uint32_t*>(&sm.Pl[ta][c0]) = lo;
                    split2(v2, v3, hi, lo);
                    *reinterpret_cast<uint32_t*>(&sm.Ph[tb][c0]) = hi;
                    *reinterpret_cast<uint32_t*>(&sm.Pl[tb][c0]) = lo;
                }
            }
        }
        // what the state at the chunk's start gives
        float o[4][2][4];
#pragma unroll
        for (int m = 0; m < 4; ++m)
#pragma unroll
            for (int j = 0; j < 2; ++j) o[m][j][0] = o[m][j][1] = o[m][j][2] = o[m][j][3] = 0.f;
        const bool first = t0 == 0 && fresh;
        if (!first) {
#pragma unroll
            for (int kk = 0; kk < NT; ++kk) {
                uint32_t h0, h1, h2, h3, l0, l1, l2, l3;
                split2(s[2 * kk][0], s[2 * kk][1], h0, l0);
                split2(s[2 * kk + 1][0], s[2 * kk + 1][1], h1, l1);
                split2(s[2 * kk][2], s[2 * kk][3], h2, l2);
                split2(s[2 * kk + 1][2], s[2 * kk + 1][3], h3, l3);
#pragma unroll
                for (int m = 0; m < 4; ++m) {
                    uint32_t af[4];
                    mma::ldsm_x4(af, c_addr + ((m * 16 + (lane & 15)) * Sm::LDN + kk * 16 + (lane >> 4) * 8) * 2);
                    mma::mma16816(o[m][0], af, h0, h1);
                    mma::mma16816(o[m][1], af, h2, h3);
                    mma::mma16816(o[m][0], af, l0, l1);
                    mma::mma16816(o[m][1], af, l2, l3);
                }
            }
#pragma unroll
            for (int m = 0; m < 4; ++m) {
                const float ea = expf(sm.cum[m * 16 + qr]), eb = expf(sm.cum[m * 16 + qr + 8]);
#pragma unroll
                for (int j = 0; j < 2; ++j) o[m][j][0] *= ea, o[m][j][1] *= ea, o[m][j][2] *= eb, o[m][j][3] *= eb;
            }
        }
        __syncthreads();                                          // the score tile is complete
        // the chunk's own tokens, and the update of the state: x as B operand / its scaled transpose as A operand
        const float cum_l = sm.cum[CL - 1];
        const float dl = expf(cum_l);
#pragma unroll
        for (int j = 0; j < 2 * NT; ++j) s[j][0] *= dl, s[j][1] *= dl, s[j][2] *= dl, s[j][3] *= dl;
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) {
            uint32_t xf[4];                                       // k = token, two 8-column blocks
            mma::ldsm_x4_t(xf, x_addr + ((ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * Sm::LDP + warp * 16 + (lane >> 4) * 8) * 2);
#pragma unroll
            for (int m = 0; m < 4; ++m) {
                if (m >= ks) {
                    uint32_t af[4];
                    const uint32_t off = ((m * 16 + (lane & 15)) * Sm::LDS + ks * 16 + (lane >> 4) * 8) * 2;
                    mma::ldsm_x4(af, ph_addr + off);
                    mma::mma16816(o[m][0], af, xf[0], xf[1]);
                    mma::mma16816(o[m][1], af, xf[2], xf[3]);
                    mma::ldsm_x4(af, pl_addr + off);
                    mma::mma16816(o[m][0], af, xf[0], xf[1]);
                    mma::mma16816(o[m][1], af, xf[2], xf[3]);
                }
            }
            // rows = columns of x, k = token: {rows 0-7, 8-15} x {tokens 0-7, 8-15}
            uint32_t xt[4], ah[4], al[4];
            mma::ldsm_x4_t(xt, x_addr + ((ks * 16 + (lane & 7) + (lane >> 4) * 8) * Sm::LDP + warp * 16 + ((lane >> 3) & 1) * 8) * 2);
            const int s0 = ks * 16 + qc;
            const float w0 = expf(cum_l - sm.cum[s0]) * sm.dt[s0], w1 = expf(cum_l - sm.cum[s0 + 1]) * sm.dt[s0 + 1];
            const float w2 = expf(cum_l - sm.cum[s0 + 8]) * sm.dt[s0 + 8], w3 = expf(cum_l - sm.cum[s0 + 9]) * sm.dt[s0 + 9];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float2 v = unpack2(xt[i]);
                split2(v.x * (i < 2 ? w0 : w2), v.y * (i < 2 ? w1 : w3), ah[i], al[i]);
            }
#pragma unroll
            for (int j = 0; j < NT; ++j) {
                uint32_t bf[4];
                mma::ldsm_x4_t(bf, b_addr + ((ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * Sm::LDN + j * 16 + (lane >> 4) * 8) * 2);
                mma::mma16816(s[2 * j], ah, bf[0], bf[1]);
                mma::mma16816(s[2 * j + 1], ah, bf[2], bf[3]);
                mma::mma16816(s[2 * j], al, bf[0], bf[1]);
                mma::mma16816(s[2 * j + 1], al, bf[2], bf[3]);
            }
        }
        // store, with the skip term
#pragma unroll
        for (int m = 0; m < 4; ++m)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int t = m * 16 + qr + e * 8;
                if (t0 + t < n) {
#pragma unroll
                    for (int j = 0; j < 2; ++j) {
                        const int p = pw + j * 8 + qc;
                        if (p < P) {                              // P is even here
                            const float2 xv = unpack2(*reinterpret_cast<const uint32_t*>(&sm.X[k][t][warp * 16 + j * 8 + qc]));
                            float v[2] = {fmaf(dsk, xv.x, o[m][j][2 * e]), fmaf(dsk, xv.y, o[m][j][2 * e + 1])};
                            TY* dst = y + ((row0 + t0 + t) * H + h) * P + p;
                            if (sizeof(TY) == 4) *reinterpret_cast<float2*>(dst) = make_float2(v[0], v[1]);
                            else *reinterpret_cast<uint32_t*>(dst) = mma::pack2(v[0], v[1]);
                        }
                    }
                }
            }
        __syncthreads();                                          // buffer k, the score tile and the sums are free again
    }
#pragma unroll
    for (int j = 0; j < 2 * NT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = j * 8 + qc + (e & 1), p = pw + qr + (e >> 1) * 8;
            if (i < N && p < P) Sg[(long long)i * P + p] = s[j][e];
        }
}

// ---- gate and grouped norm -------------------------------------------------------------------------------------------------
// One CTA per (row, group of gs columns): v = y act(z);  out = v / sqrt(mean(v^2) + eps) * w  (w over all columns).
template <typename TY, typename T, int VEC>
__global__ void gate_norm_kernel(const TY* __restrict__ y, long long ld_y, const T* __restrict__ z, long long ld_z,
                                 const float* __restrict__ w, T* __restrict__ out, long long ld_out, int gs, float eps, int act) {
    constexpr int RV = 4;                    // column groups per thread that stay in registers
    __shared__ float red[32];
    const long long row = blockIdx.x;
    const int c0 = blockIdx.y * gs;
    const TY* yr = y + row * ld_y + c0;
    const T* zr = z + row * ld_z + c0;
    T* orow = out + row * ld_out + c0;
    float v[RV][VEC], ss = 0.f;
    auto gated = [&](int c, float* t) {
        float g[VEC];
        ldv<VEC>(yr + c, t);
        ldv<VEC>(zr + c, g);
#pragma unroll
        for (int i = 0; i < VEC; ++i) t[i] *= act == 1 ? ScanMath<T>::silu(g[i]) : ScanMath<T>::sigmoid(g[i]);
    };
#pragma unroll
    for (int k = 0; k < RV; ++k) {
        const int c = (threadIdx.x + k * blockDim.x) * VEC;
        if (c < gs) {
            gated(c, v[k]);
#pragma unroll
            for (int i = 0; i < VEC; ++i) ss = fmaf(v[k][i], v[k][i], ss);
        }
    }
    for (int c = (threadIdx.x + RV * blockDim.x) * VEC; c < gs; c += blockDim.x * VEC) {
        float t[VEC];
        gated(c, t);
#pragma unroll
        for (int i = 0; i < VEC; ++i) ss = fmaf(t[i], t[i], ss);
    }
    const float r = 1.f / sqrtf(block_sum(ss, red) / (float)gs + eps);
    auto store = [&](int c, float* t) {
        float g[VEC];
        ldv<VEC>(w + c0 + c, g);
#pragma unroll
        for (int i = 0; i < VEC; ++i) g[i] *= t[i] * r;
        stv<VEC>(orow + c, g);
    };
#pragma unroll
    for (int k = 0; k < RV; ++k) {
        const int c = (threadIdx.x + k * blockDim.x) * VEC;
        if (c < gs) store(c, v[k]);
    }
    for (int c = (threadIdx.x + RV * blockDim.x) * VEC; c < gs; c += blockDim.x * VEC) {
        float t[VEC];
        gated(c, t);
        store(c, t);
    }
}

template <typename TY, typename T>
int launch_gate(const void* y, long long ld_y, const void* z, long long ld_z, const float* w, void* out, long long ld_out,
                long long rows, int n, int groups, float eps, int act, bool vec, cudaStream_t st) {
    const int gs = n / groups, per = vec ? 4 : 1;
    int threads = 32;
    while (threads < 256 && threads * per * 2 < gs) threads <<= 1;
    dim3 grid((unsigned)rows, groups);
    if (vec) gate_norm_kernel<TY, T, 4><<<grid, threads, 0, st>>>((const TY*)y, ld_y, (const T*)z, ld_z, w, (T*)out, ld_out, gs, eps, act);
    else gate_norm_kernel<TY, T, 1><<<grid, threads, 0, st>>>((const TY*)y, ld_y, (const T*)z, ld_z, w, (T*)out, ld_out, gs, eps, act);
    NXD_LAUNCH_CHECK();
    return 0;
}

}  // namespace

// dtypes: 0 bf16, 1 fp32.  proj [B * Tn, ld] points at the first of the C channels; conv_w fp32 [taps, C] (last row = the
// current token), bias fp32 [C] or NULL; conv_state fp32 [lines, taps - 1, C], moved to the end of the step (zeros before
// the start of the sequence; rows without real tokens keep theirs).  out [B * Tn, ld_out]: silu(convolution), zeros in padding
// rows.  q_start [B], n_new [B] or NULL, seq_ids [B] or NULL as in the attention entry points.
NXD_API int nxd_conv_silu(int dtype, int out_dtype, const void* proj, long long ld, const float* conv_w, const float* bias,
                          float* conv_state, void* out, long long ld_out, const int* q_start, const int* n_new,
                          const int* seq_ids, int B, int Tn, int C, int taps, void* stream) {
    if ((long long)B * Tn * C == 0) return 0;
    NXD_REQUIRE(taps >= 1, "short convolution with %d taps", taps);
    NXD_REQUIRE(B < 65536, "short convolution: %d rows", B);
    cudaStream_t st = (cudaStream_t)stream;
    auto al = [](const void* p) { return ((uintptr_t)p % 16) == 0; };
    const bool vec = C % 4 == 0 && ld % 4 == 0 && ld_out % 4 == 0 && al(proj) && al(out) && al(conv_state);
    // few tokens: one thread walks the whole step and moves the state itself
    const int TT = Tn <= 64 ? Tn : 32, move = Tn <= 64 ? 1 : 0;
    const bool wide = vec && !move && dtype == 0 && out_dtype == 0 && taps == 4 && C % 8 == 0 && ld % 8 == 0 && ld_out % 8 == 0 &&
                      al(conv_w) && al(bias);
    const int width = 128 * (wide ? 8 : (vec ? 4 : 1)), tokens = wide ? STRIP : TT;
    dim3 grid((C + width - 1) / width, (Tn + tokens - 1) / tokens, B);
    NXD_REQUIRE(grid.y < 65536, "short convolution: %d tokens", Tn);
#define NXD_CONV(T, TO, V, K)                                                                                            \
    conv_silu_kernel<T, TO, V, K><<<grid, 128, 0, st>>>((const T*)proj, ld, conv_w, bias, conv_state, (TO*)out, ld_out,    \
                                                        q_start, n_new, seq_ids, Tn, C, taps, TT, move)
#define NXD_CONV_T(T, TO)                                                                                                \
    do {                                                                                                                 \
        if (taps == 4) { if (vec) NXD_CONV(T, TO, 4, 4); else NXD_CONV(T, TO, 1, 4); }                                    \
        else { if (vec) NXD_CONV(T, TO, 4, 0); else NXD_CONV(T, TO, 1, 0); }                                              \
    } while (0)
    if (wide)
        conv_silu_strip_kernel<4><<<grid, 128, 0, st>>>((const bf16*)proj, ld, conv_w, bias, conv_state, (bf16*)out, ld_out,
                                                        q_start, n_new, seq_ids, Tn, C);
    else if (dtype == 0 && out_dtype == 0) NXD_CONV_T(bf16, bf16);
    else if (dtype == 0) NXD_CONV_T(bf16, float);
    else { NXD_REQUIRE(out_dtype == 1, "short convolution: fp32 input, 16-bit output"); NXD_CONV_T(float, float); }
#undef NXD_CONV_T
#undef NXD_CONV
    NXD_LAUNCH_CHECK();
    if (!move && taps > 1) {
        dim3 g2((C + 127) / 128, B);
        if (dtype == 0) conv_state_kernel<bf16><<<g2, 128, 0, st>>>((const bf16*)proj, ld, conv_state, q_start, n_new, seq_ids, Tn, C, taps);
        else conv_state_kernel<float><<<g2, 128, 0, st>>>((const float*)proj, ld, conv_state, q_start, n_new, seq_ids, Tn, C, taps);
        NXD_LAUNCH_CHECK();
    }
    return 0;
}

// x, z, out [B * Tn, ...] (dtype), dt fp32 pre-activations [B * Tn, ld_dt] (softplus(dt + dt_bias) is taken here), bc fp32
// [B * Tn, ld_bc]: B at column b_off, C at c_off (N each); a_log fp32 [C, N], dskip fp32 [C]; S fp32 [lines, C, N] in place.
NXD_API int nxd_selective_scan(int dtype, const void* x, long long ld_x, const float* dt, long long ld_dt, const float* dt_bias,
                               const float* bc, long long ld_bc, int b_off, int c_off, const void* z, long long ld_z,
                               const float* a_log, const float* dskip, float* S, void* out, long long ld_out,
                               const int* q_start, const int* n_new, const int* seq_ids, int B, int Tn, int C, int N,
                               void* stream) {
    if ((long long)B * Tn * C == 0) return 0;
    NXD_REQUIRE(N >= 1 && N <= 512, "selective scan: %d states per channel", N);
    NXD_REQUIRE(B < 65536, "selective scan: %d rows", B);
    cudaStream_t st = (cudaStream_t)stream;
#define NXD_SEL(T, NS_, R_, CPT_, TS_)                                                                                   \
    return launch_selective<T, NS_, R_, CPT_, TS_>(x, ld_x, dt, ld_dt, dt_bias, bc, ld_bc, b_off, c_off, z, ld_z, a_log,  \
                                                   dskip, S, out, ld_out, q_start, n_new, seq_ids, B, Tn, C, N, st)
#define NXD_SEL_T(T)                                                                                                     \
    do {                                                                                                                 \
        if (N <= 4) NXD_SEL(T, 4, 1, 1, 16);                                                                             \
        if (N <= 8) NXD_SEL(T, 4, 2, 2, 16);                                                                             \
        if (N <= 16) NXD_SEL(T, 4, 4, 2, 16);                                                                            \
        if (N <= 32) NXD_SEL(T, 8, 4, 1, 16);                                                                            \
        if (N <= 64) NXD_SEL(T, 8, 8, 1, 16);                                                                            \
        if (N <= 128) NXD_SEL(T, 16, 8, 1, 16);                                                                          \
        if (N <= 256) NXD_SEL(T, 32, 8, 1, 8);                                                                           \
        NXD_SEL(T, 64, 8, 1, 8);                                                                                         \
    } while (0)
    if (dtype == 0) NXD_SEL_T(bf16);
    NXD_SEL_T(float);
#undef NXD_SEL_T
#undef NXD_SEL
}

// One token per row of the same recurrence; the step sizes' pre-activations are the first `rank` columns of p (fp32 [B, ld_p], B and C
// at b_off and c_off) times dt_w [C, rank] (dtype; rank a multiple of 8).
NXD_API int nxd_selective_step(int dtype, const void* x, long long ld_x, const void* dt_w, int rank, const float* dt_bias,
                               const float* p, long long ld_p, int b_off, int c_off, const void* z, long long ld_z,
                               const float* a_log, const float* dskip, float* S, void* out, long long ld_out,
                               const int* q_start, const int* seq_ids, int B, int C, int N, void* stream) {
    if ((long long)B * C == 0) return 0;
    auto al = [](const void* q) { return ((uintptr_t)q % 16) == 0; };
    NXD_REQUIRE(rank % 8 == 0 && al(dt_w), "selective scan: step sizes of rank %d", rank);
    const size_t smem = (size_t)STEP_ROWS * ((rank + 2 * N + 3) & ~3) * sizeof(float);
    NXD_REQUIRE(N >= 1 && smem <= 48 * 1024, "selective scan: rank %d, %d states", rank, N);
    dim3 grid((C + 31) / 32, (B + STEP_ROWS - 1) / STEP_ROWS);
    NXD_REQUIRE(grid.y < 65536, "selective scan: %d rows", B);
    const bool vec = N % 4 == 0 && al(S) && al(a_log);
    cudaStream_t st = (cudaStream_t)stream;
#define NXD_SSTEP(T, V)                                                                                                  \
    selective_step_kernel<T, V><<<grid, STEP_THREADS, smem, st>>>((const T*)x, ld_x, (const T*)dt_w, rank, dt_bias, p, ld_p, \
                                                                  b_off, c_off, (const T*)z, ld_z, a_log, dskip, S, (T*)out, \
                                                                  ld_out, q_start, seq_ids, B, C, N)
    if (dtype == 0) { if (vec) NXD_SSTEP(bf16, true); else NXD_SSTEP(bf16, false); }
    else { if (vec) NXD_SSTEP(float, true); else NXD_SSTEP(float, false); }
#undef NXD_SSTEP
    NXD_LAUNCH_CHECK();
    return 0;
}

// xbc [B * Tn, ld] (dtype): x [H, P] at column x_off, B and C [G, N] at b_off and c_off (after the convolution); dt fp32
// pre-activations [B * Tn, ld_dt], one per head; dt_bias (or NULL), a_log, dskip fp32 [H]; S fp32 [lines, H, N, P] in place;
// y [B * Tn, H, P] (y_dtype).  dt NULL (one token per row): the pre-activations are hin [B, W] times the rows of dt_w [H, W], both
// of the type of xbc.  impl: 0 choose, 1 token by token, 2 chunks on the tensor cores (an error where they do not apply).
NXD_API int nxd_state_space_heads(int dtype, int y_dtype, const void* xbc, long long ld, int x_off, int b_off, int c_off,
                                  const float* dt, long long ld_dt, const float* dt_bias, const float* a_log,
                                  const float* dskip, float* S, void* y, const int* q_start, const int* n_new,
                                  const int* seq_ids, int B, int Tn, int H, int G, int N, int P, int impl,
                                  const void* hin, const void* dt_w, int W, void* stream) {
    if ((long long)B * Tn * H * P == 0) return 0;
    NXD_REQUIRE(G > 0 && H % G == 0, "state-space heads: %d heads over %d groups", H, G);
    NXD_REQUIRE(N >= 1 && N <= 1024, "state-space heads: state size %d", N);
    NXD_REQUIRE(B < 65536 && H < 65536, "state-space heads: %d rows of %d heads", B, H);
    NXD_REQUIRE(y_dtype == 1 || y_dtype == dtype, "state-space heads: output type");
    cudaStream_t st = (cudaStream_t)stream;
    auto al = [](const void* p) { return ((uintptr_t)p % 16) == 0; };
    const bool single = Tn == 1 && n_new == nullptr && impl == 0;
    NXD_REQUIRE(dt != nullptr || (single && hin != nullptr && dt_w != nullptr), "state-space heads: %s", "no step sizes");
    NXD_REQUIRE(dt != nullptr || W % 8 != 0 || (al(hin) && al(dt_w)), "state-space heads: %s", "unaligned inputs of the step sizes");
    if (single) {
        const bool vec = P % 4 == 0 && al(S);
        dim3 grid((P + 31) / 32, H, B);
        const size_t smem = (size_t)2 * N * sizeof(float);
#define NXD_STEP(T, TY, V)                                                                                               \
    ssd_step_kernel<T, TY, V><<<grid, 128, smem, st>>>((const T*)xbc, ld, x_off, b_off, c_off, dt, ld_dt, dt_bias, a_log, \
                                                       dskip, S, (TY*)y, q_start, seq_ids, H, G, N, P, (const T*)hin, (const T*)dt_w, W)
        if (dtype == 1) { if (vec) NXD_STEP(float, float, 4); else NXD_STEP(float, float, 1); }
        else if (y_dtype == 1) { if (vec) NXD_STEP(bf16, float, 4); else NXD_STEP(bf16, float, 1); }
        else { if (vec) NXD_STEP(bf16, bf16, 4); else NXD_STEP(bf16, bf16, 1); }
#undef NXD_STEP
        NXD_LAUNCH_CHECK();
        return 0;
    }
    const bool chunks = dtype == 0 && N <= 128 && N % 8 == 0 && P % 8 == 0 && ld % 8 == 0 && x_off % 8 == 0 && b_off % 8 == 0 &&
                        c_off % 8 == 0 && al(xbc) && al(y);
    NXD_REQUIRE(impl != 2 || chunks, "state-space heads: the chunk form does not apply (state %d, head size %d)", N, P);
    if (impl == 2 || (impl == 0 && chunks && Tn >= CL)) {
#define NXD_CHUNK(TY, NT_, W_)                                                                                           \
    do {                                                                                                                 \
        auto kern = ssd_chunk_kernel<TY, NT_, W_>;                                                                       \
        const size_t smem = sizeof(ChunkSmem<NT_, W_>);                                                                  \
        if (smem > 48 * 1024)                                                                                            \
            NXD_CHECK_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));          \
        dim3 grid((P + 16 * W_ - 1) / (16 * W_), H, B);                                                                  \
        kern<<<grid, W_ * 32, smem, st>>>((const bf16*)xbc, ld, x_off, b_off, c_off, dt, ld_dt, dt_bias, a_log, dskip, S, \
                                          (TY*)y, q_start, n_new, seq_ids, Tn, H, G, N, P);                               \
    } while (0)
#define NXD_CHUNK_N(TY, W_)                                                                                              \
    do { if (N <= 32) NXD_CHUNK(TY, 2, W_); else if (N <= 64) NXD_CHUNK(TY, 4, W_); else NXD_CHUNK(TY, 8, W_); } while (0)
        // heads of at most 32 columns, and grids that would leave half the GPU idle, take the narrow slices
        const bool narrow = P <= 32 || (long long)B * H * ((P + 63) / 64) * 2 <= nxd_num_sms();
        if (y_dtype == 1) { if (narrow) NXD_CHUNK_N(float, 2); else NXD_CHUNK_N(float, 4); }
        else { if (narrow) NXD_CHUNK_N(bf16, 2); else NXD_CHUNK_N(bf16, 4); }
#undef NXD_CHUNK_N
#undef NXD_CHUNK
        NXD_LAUNCH_CHECK();
        return 0;
    }
    const int npt = N <= 32 ? 8 : (N <= 64 ? 16 : 32);
    int R = 1;
    while (R * npt < N) R <<= 1;
    const int CT = 128 / R;
    const size_t smem = (size_t)16 * (2 * R * (npt + 4) + CT) * sizeof(float);
    dim3 grid((P + CT - 1) / CT, H, B);
#define NXD_SCAN(T, TY, N_)                                                                                              \
    do {                                                                                                                 \
        auto kern = ssd_scan_kernel<T, TY, N_>;                                                                          \
        if (smem > 48 * 1024)                                                                                            \
            NXD_CHECK_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));          \
        kern<<<grid, 128, smem, st>>>((const T*)xbc, ld, x_off, b_off, c_off, dt, ld_dt, dt_bias, a_log, dskip, S, (TY*)y, \
                                      q_start, n_new, seq_ids, Tn, H, G, N, P, R);                                        \
    } while (0)
#define NXD_SCAN_T(T, TY) do { if (npt == 8) NXD_SCAN(T, TY, 8); else if (npt == 16) NXD_SCAN(T, TY, 16); else NXD_SCAN(T, TY, 32); } while (0)
    if (dtype == 1) NXD_SCAN_T(float, float);
    else if (y_dtype == 1) NXD_SCAN_T(bf16, float);
    else NXD_SCAN_T(bf16, bf16);
#undef NXD_SCAN_T
#undef NXD_SCAN
    NXD_LAUNCH_CHECK();
    return 0;
}

// y [rows, ld_y] (y_dtype: 0 bf16, 1 fp32), z and out [rows, ...] (dtype): v = y act(z) (act 0 sigmoid, 1 silu), every one of the
// groups of n / groups columns divided by sqrt(mean(v^2) + eps), times w fp32 [n].
NXD_API int nxd_gate_norm(int y_dtype, int dtype, const void* y, long long ld_y, const void* z, long long ld_z, const float* w,
                          void* out, long long ld_out, long long rows, int n, int groups, float eps, int act, void* stream) {
    if (rows * n == 0) return 0;
    NXD_REQUIRE(rows < (1ll << 31), "gate: %lld rows", rows);
    NXD_REQUIRE(groups > 0 && n % groups == 0 && groups < 65536, "gate: %d columns in %d groups", n, groups);
    NXD_REQUIRE(dtype == 0 || y_dtype == 1, "gate: %s", "16-bit input, fp32 gate");
    auto al = [](const void* p) { return ((uintptr_t)p % 16) == 0; };
    const bool vec = (n / groups) % 4 == 0 && ld_y % 4 == 0 && ld_z % 4 == 0 && ld_out % 4 == 0 && al(y) && al(z) && al(out) && al(w);
    cudaStream_t st = (cudaStream_t)stream;
    if (dtype == 1) return launch_gate<float, float>(y, ld_y, z, ld_z, w, out, ld_out, rows, n, groups, eps, act, vec, st);
    if (y_dtype == 1) return launch_gate<float, bf16>(y, ld_y, z, ld_z, w, out, ld_out, rows, n, groups, eps, act, vec, st);
    return launch_gate<bf16, bf16>(y, ld_y, z, ld_z, w, out, ld_out, rows, n, groups, eps, act, vec, st);
}
