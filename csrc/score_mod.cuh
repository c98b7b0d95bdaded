// What an attention kernel may do to a score after the scaled product, next to the mask and the linear distance bias, and to
// the head output after the value product:
//
//   soft cap         s <- cap * tanh(s / cap)                                        (cap > 0)
//   log distance     s <- s - r1_h * ln(1 + r2_h * (i - j))                          (r1, r2 != NULL)
//   sigmoid weights  weight = sigmoid(s + pb_h), not normalised over the keys        (pb != NULL; no softmax, no sink)
//   output gate      o <- o * sigmoid(gate[row, h])                                  (gate != NULL; one number per head)
//                    o[c] <- o[c] * sigmoid(gate[row, h, c]) * gate_mul                 (gate_cols > 0: one number per element)
//
// tanh in fp32 for |x| < 0.4 is the odd power series up to x^9 (next term below 1e-6 of the value), beyond that
// 1 - 2 / (1 + exp(2 |x|)); the kernels choose once per tile where they can.  The fp32 kernels take two more terms of the series
// and a rounded division: a cap of 20 turns an error of 1e-6 in tanh into one of 2e-5 in the weight.
#pragma once
#include "common.cuh"

struct ScoreMod {
    float cap;
    const float* r1;
    const float* r2;
    const float* pb;
    const void* gate;        // activation dtype; pre-activation of (row n, head h) at gate[n * gate_ld + h]
    long long gate_ld;
    int gate_cols;           // > 0: value size; pre-activation of (row n, head h, column c) at gate[n * gate_ld + h * gate_cols + c]
    float gate_mul;          // of the gate per element
    long long out_ld;        // elements between output rows (0: the heads of a row are all there is in it)
    __host__ __device__ int mode() const { return pb != nullptr ? 2 : ((cap > 0.f || r1 != nullptr) ? 1 : 0); }
};

namespace score {

constexpr float kSeriesLimit = 0.4f;
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float tanh_series(float x) {
    const float z = x * x;
    float p = fmaf(z, 62.f / 2835.f, -17.f / 315.f);
    p = fmaf(z, p, 2.f / 15.f);
    p = fmaf(z, p, -1.f / 3.f);
    return fmaf(x * z, p, x);
}
__device__ __forceinline__ float tanh_exp(float x) {
    const float e = exp2f(2.f * kLog2e * fabsf(x));
    return copysignf(1.f - __fdividef(2.f, 1.f + fminf(e, 1e30f)), x);
}
__device__ __forceinline__ float tanh_any(float x) { return fabsf(x) < kSeriesLimit ? tanh_series(x) : tanh_exp(x); }
// to the last bits of fp32, also where the compiler may approximate exponentials and divisions: the exponent 2 |x| log2(e) is
// split into its nearest integer and a remainder taken with fused multiply-adds, so that its rounding does not enter
__device__ __forceinline__ float tanh_fp32(float x) {
    const float a = fabsf(x);
    if (a < kSeriesLimit) {
        const float z = x * x;
        float p = fmaf(z, 21844.f / 6081075.f, -1382.f / 155925.f);
        p = fmaf(z, p, 62.f / 2835.f);
        p = fmaf(z, p, -17.f / 315.f);
        p = fmaf(z, p, 2.f / 15.f);
        p = fmaf(z, p, -1.f / 3.f);
        return fmaf(x * z, p, x);
    }
    const float b = fminf(2.f * a, 40.f), n = rintf(b * kLog2e);
    const float e = exp2f(n) * exp2f(fmaf(b, kLog2e, -n));
    return copysignf(1.f - __fdiv_rn(2.f, 1.f + e), x);
}

// sigmoid(x) for x given in log2 units (x * log2 e); the clamp keeps 1 + 2^-x finite
__device__ __forceinline__ float sigmoid_log2(float x2) { return __fdividef(1.f, 1.f + exp2f(fminf(-x2, 100.f))); }
__device__ __forceinline__ float sigmoid(float x) { return sigmoid_log2(x * kLog2e); }

__device__ __forceinline__ float ldg(const float* p) { return *p; }
__device__ __forceinline__ float ldg(const bf16* p) { return __bfloat162float(*p); }
template <typename T>
__device__ __forceinline__ float out_gate(const ScoreMod& m, long long row, int h) {
    return (m.gate == nullptr || m.gate_cols > 0) ? 1.f : sigmoid(ldg(reinterpret_cast<const T*>(m.gate) + row * m.gate_ld + h));
}

template <typename T>
__device__ __forceinline__ float elem_gate(const ScoreMod& m, long long row, int h, int c) {
    return m.gate_cols <= 0 ? 1.f : m.gate_mul * sigmoid(ldg(reinterpret_cast<const T*>(m.gate) + row * m.gate_ld + (long long)h * m.gate_cols + c));
}
// two neighbouring columns (c even) of a 16-bit gate
__device__ __forceinline__ float2 elem_gate2(const ScoreMod& m, long long row, int h, int c) {
    if (m.gate_cols <= 0) return make_float2(1.f, 1.f);
    const bf16* p = reinterpret_cast<const bf16*>(m.gate) + row * m.gate_ld + (long long)h * m.gate_cols + c;
    return make_float2(m.gate_mul * sigmoid(ldg(p)), m.gate_mul * sigmoid(ldg(p + 1)));
}
__device__ __forceinline__ long long out_pitch(const ScoreMod& m, int columns) { return m.out_ld > 0 ? m.out_ld : columns; }

}  // namespace score
