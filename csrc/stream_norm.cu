// The fp32 residual stream of plain pre-norm decoders.
//
//   embed_norm      x = e / sqrt(mean(e^2) + eps) * w_embed,  e = table[token] (+ position vector);  h = norm(x) * w_next
//                   position vector: entry 2 i = sin(p f_i), entry 2 i + 1 = cos(p f_i), f_i = base^(-2 i / W)
//   residual_norm   x <- x + y (+ bias);   h = cast(x / sqrt(mean(x^2) + eps) * w_next)
//   stream_update   x <- [x] + scale * (y + bias) + mul * table[token] + shift, any of the terms, and the same norm: the entry of a
//                   model (no x yet), a sublayer with a layer scale, the start of a pass of a looped range of layers
//
// One CTA per token; the row stays in registers between the passes (up to RV groups of VEC columns per thread; wider rows are
// read again), statistics in fp32.  Angles are reduced in double precision, so positions of any size keep the accuracy of
// the fp32 sine and cosine.  This file is compiled without fast-math.
#include "common.cuh"

namespace {

template <int VEC>
__device__ __forceinline__ void ldv(const float* p, float* v) {
    if (VEC == 4) {
        const float4 t = *reinterpret_cast<const float4*>(p);
        v[0] = t.x, v[1] = t.y, v[2] = t.z, v[3] = t.w;
    } else {
        v[0] = *p;
    }
}
template <int VEC>
__device__ __forceinline__ void ldv(const bf16* p, float* v) {
    if (VEC == 4) {
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
    if (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else *p = v[0];
}
template <int VEC>
__device__ __forceinline__ void stv(bf16* p, const float* v) {
    if (VEC == 4) {
        uint2 raw;
        *reinterpret_cast<bf162*>(&raw.x) = __floats2bfloat162_rn(v[0], v[1]);
        *reinterpret_cast<bf162*>(&raw.y) = __floats2bfloat162_rn(v[2], v[3]);
        *reinterpret_cast<uint2*>(p) = raw;
    } else {
        *p = __float2bfloat16_rn(v[0]);
    }
}

constexpr int RV = 4;            // column groups per thread that stay in registers

// the further terms of a stream update
struct StreamTerms {
    const float* scale;          // [W], times (y + bias)
    const float* shift;          // [W]
    const void* table;           // [vocab, W], bf16 or fp32, times mul
    const long long* ids;        // [rows]
    float mul;
    int vocab, table_fp32, init; // init: x holds nothing yet
};

template <typename TY, typename TH, int VEC, int NT, bool TERMS>
__global__ void __launch_bounds__(NT)
residual_norm_kernel(float* __restrict__ x, const TY* __restrict__ y, const float* __restrict__ bias,
                     const float* __restrict__ w, TH* __restrict__ h, int W, float eps, const StreamTerms ex) {
    __shared__ float red[32];
    const long long row = blockIdx.x;
    float* xr = x + row * W;
    const TY* yr = y != nullptr ? y + row * W : nullptr;
    float v[RV][VEC];
    float ss = 0.f;
    long long trow = 0;
    if (TERMS && ex.table != nullptr) trow = min(max(ex.ids[row], 0ll), (long long)ex.vocab - 1) * W;
    auto load_terms = [&](int c, float* t) {
        float a[VEC], b[VEC];
        if (ex.init) {
#pragma unroll
            for (int i = 0; i < VEC; ++i) t[i] = 0.f;
        } else {
            ldv<VEC>(xr + c, t);
        }
        if (yr != nullptr) {
            ldv<VEC>(yr + c, a);
            if (bias != nullptr) {
                ldv<VEC>(bias + c, b);
#pragma unroll
                for (int i = 0; i < VEC; ++i) a[i] += b[i];
            }
            if (ex.scale != nullptr) {
                ldv<VEC>(ex.scale + c, b);
#pragma unroll
                for (int i = 0; i < VEC; ++i) a[i] *= b[i];
            }
#pragma unroll
            for (int i = 0; i < VEC; ++i) t[i] += a[i];
        }
        if (ex.table != nullptr) {
            if (ex.table_fp32) ldv<VEC>((const float*)ex.table + trow + c, a);
            else ldv<VEC>((const bf16*)ex.table + trow + c, a);
#pragma unroll
            for (int i = 0; i < VEC; ++i) t[i] = fmaf(a[i], ex.mul, t[i]);
        }
        if (ex.shift != nullptr) {
            ldv<VEC>(ex.shift + c, a);
#pragma unroll
            for (int i = 0; i < VEC; ++i) t[i] += a[i];
        }
        stv<VEC>(xr + c, t);
#pragma unroll
        for (int i = 0; i < VEC; ++i) ss = fmaf(t[i], t[i], ss);
    };
    auto load = [&](int c, float* t) {
        if (TERMS) {
            load_terms(c, t);
            return;
        }
        ldv<VEC>(xr + c, t);
        if (yr != nullptr) {
            float a[VEC];
            ldv<VEC>(yr + c, a);
#pragma unroll
            for (int i = 0; i < VEC; ++i) t[i] += a[i];
            if (bias != nullptr) {
                ldv<VEC>(bias + c, a);
#pragma unroll
                for (int i = 0; i < VEC; ++i) t[i] += a[i];
            }
            stv<VEC>(xr + c, t);
        }
#pragma unroll
        for (int i = 0; i < VEC; ++i) ss = fmaf(t[i], t[i], ss);
    };
#pragma unroll
    for (int k = 0; k < RV; ++k) {
        const int c = (threadIdx.x + k * NT) * VEC;
        if (c < W) load(c, v[k]);
    }
    for (int c = (threadIdx.x + RV * NT) * VEC; c < W; c += NT * VEC) {
        float t[VEC];
        load(c, t);
    }
    if (w == nullptr || h == nullptr) return;
    const float r = 1.f / sqrtf(block_sum(ss, red) / (float)W + eps);
    TH* hr = h + row * W;
    auto store = [&](int c, const float* t) {
        float g[VEC];
        ldv<VEC>(w + c, g);
#pragma unroll
        for (int i = 0; i < VEC; ++i) g[i] *= t[i] * r;
        stv<VEC>(hr + c, g);
    };
#pragma unroll
    for (int k = 0; k < RV; ++k) {
        const int c = (threadIdx.x + k * NT) * VEC;
        if (c < W) store(c, v[k]);
    }
    for (int c = (threadIdx.x + RV * NT) * VEC; c < W; c += NT * VEC) {
        float t[VEC];
        ldv<VEC>(xr + c, t);
        store(c, t);
    }
}

// sine / cosine entries of two neighbouring columns (2 i, 2 i + 1) at position p; freq [ceil(W / 2)] in double
__device__ __forceinline__ void position_pair(double p, double f, float& s, float& c) {
    double a = p * f;
    a -= rint(a * 0.15915494309189535) * 6.283185307179586;
    sincosf((float)a, &s, &c);
}

template <typename TE, typename TH, int NT>
__global__ void __launch_bounds__(NT)
embed_norm_kernel(const TE* __restrict__ table, const long long* __restrict__ ids, const long long* __restrict__ pos,
                  const double* __restrict__ freq, const float* __restrict__ w_embed, const float* __restrict__ w_next,
                  float* __restrict__ x, TH* __restrict__ h, int W, int vocab, float eps) {
    extern __shared__ float rowbuf[];
    __shared__ float red[32];
    const long long row = blockIdx.x;
    const long long id = min(max(ids[row], 0ll), (long long)vocab - 1);
    const TE* er = table + id * W;
    const double p = (double)pos[row];
    float ss = 0.f;
    for (int c = threadIdx.x * 2; c < W; c += NT * 2) {
        float s = 0.f, k = 0.f;
        if (freq != nullptr) position_pair(p, freq[c >> 1], s, k);
        float a[1];
        ldv<1>(er + c, a);
        const float e0 = a[0] + s;
        rowbuf[c] = e0;
        ss = fmaf(e0, e0, ss);
        if (c + 1 < W) {
            ldv<1>(er + c + 1, a);
            const float e1 = a[0] + k;
            rowbuf[c + 1] = e1;
            ss = fmaf(e1, e1, ss);
        }
    }
    float r = 1.f / sqrtf(block_sum(ss, red) / (float)W + eps);
    float* xr = x + row * W;
    ss = 0.f;
    for (int c = threadIdx.x; c < W; c += NT) {
        const float v = rowbuf[c] * r * w_embed[c];
        xr[c] = v;
        rowbuf[c] = v;
        ss = fmaf(v, v, ss);
    }
    if (w_next == nullptr || h == nullptr) return;
    r = 1.f / sqrtf(block_sum(ss, red) / (float)W + eps);
    for (int c = threadIdx.x; c < W; c += NT) {
        const float v[1] = {rowbuf[c] * r * w_next[c]};
        stv<1>(h + row * W + c, v);
    }
}

template <typename TY, typename TH, bool TERMS>
int launch_residual(float* x, const void* y, const float* bias, const float* w, void* h, long long rows, int W, float eps,
                    bool vec, const StreamTerms& ex, cudaStream_t st) {
#define NXD_RN(V, NT)                                                                                                    \
    residual_norm_kernel<TY, TH, V, NT, TERMS><<<(unsigned)rows, NT, 0, st>>>(x, (const TY*)y, bias, w, (TH*)h, W, eps, ex)
    if (vec && W <= 1024) NXD_RN(4, 64);
    else if (vec && W <= 2048) NXD_RN(4, 128);
    else if (vec) NXD_RN(4, 256);
    else NXD_RN(1, 128);
#undef NXD_RN
    NXD_LAUNCH_CHECK();
    return 0;
}

}  // namespace

// x [rows, W] fp32 stream (updated in place when y is given); y [rows, W] (y_dtype) or NULL; bias [W] fp32 or NULL (added
// with y); w [W] fp32 and h [rows, W] (h_dtype), or both NULL.  dtypes: 0 bf16, 1 fp32.
NXD_API int nxd_residual_norm(int y_dtype, int h_dtype, float* x, const void* y, const float* bias, const float* w, void* h,
                              long long rows, int W, float eps, void* stream) {
    if (rows == 0) return 0;
    NXD_REQUIRE(rows < (1ll << 31), "residual norm: %lld rows", rows);
    cudaStream_t st = (cudaStream_t)stream;
    auto al = [](const void* p) { return p == nullptr || ((uintptr_t)p % 16) == 0; };
    const bool vec = W % 4 == 0 && al(x) && al(y) && al(bias) && al(w) && al(h);
    const StreamTerms ex = {};
    switch ((y_dtype << 1) | h_dtype) {
        case 0: return launch_residual<bf16, bf16, false>(x, y, bias, w, h, rows, W, eps, vec, ex, st);
        case 1: return launch_residual<bf16, float, false>(x, y, bias, w, h, rows, W, eps, vec, ex, st);
        case 2: return launch_residual<float, bf16, false>(x, y, bias, w, h, rows, W, eps, vec, ex, st);
        default: return launch_residual<float, float, false>(x, y, bias, w, h, rows, W, eps, vec, ex, st);
    }
}

// As nxd_residual_norm with further terms: x <- (init ? 0 : x) + scale * (y + bias) + mul * table[ids] + shift.  scale and shift
// [W] fp32 or NULL; table [vocab, W] (t_dtype) with ids [rows] int64, or NULL.
NXD_API int nxd_stream_update(int y_dtype, int h_dtype, int t_dtype, float* x, const void* y, const float* bias,
                              const float* scale, const void* table, const long long* ids, float mul, int vocab,
                              const float* shift, int init, const float* w, void* h, long long rows, int W, float eps,
                              void* stream) {
    if (rows == 0) return 0;
    NXD_REQUIRE(rows < (1ll << 31), "stream update: %lld rows", rows);
    NXD_REQUIRE(table == nullptr || (ids != nullptr && vocab > 0), "stream update: a table without ids");
    cudaStream_t st = (cudaStream_t)stream;
    auto al = [](const void* p) { return p == nullptr || ((uintptr_t)p % 16) == 0; };
    const bool vec = W % 4 == 0 && al(x) && al(y) && al(bias) && al(w) && al(h) && al(scale) && al(shift) && al(table);
    StreamTerms ex;
    ex.scale = scale, ex.shift = shift, ex.table = table, ex.ids = ids, ex.mul = mul, ex.vocab = vocab, ex.table_fp32 = t_dtype;
    ex.init = init;
    switch ((y_dtype << 1) | h_dtype) {
        case 0: return launch_residual<bf16, bf16, true>(x, y, bias, w, h, rows, W, eps, vec, ex, st);
        case 1: return launch_residual<bf16, float, true>(x, y, bias, w, h, rows, W, eps, vec, ex, st);
        case 2: return launch_residual<float, bf16, true>(x, y, bias, w, h, rows, W, eps, vec, ex, st);
        default: return launch_residual<float, float, true>(x, y, bias, w, h, rows, W, eps, vec, ex, st);
    }
}

// table [vocab, W] (e_dtype), ids / pos [rows] int64, freq [ceil(W / 2)] double or NULL (no position vectors), w_embed [W]
// fp32; x [rows, W] fp32 out; w_next [W] fp32 and h [rows, W] (h_dtype), or both NULL.
NXD_API int nxd_embed_norm(int e_dtype, int h_dtype, const void* table, const long long* ids, const long long* pos,
                           const double* freq, const float* w_embed, const float* w_next, float* x, void* h, long long rows,
                           int W, int vocab, float eps, void* stream) {
    if (rows == 0) return 0;
    NXD_REQUIRE(rows < (1ll << 31), "embedding: %lld rows", rows);
    const size_t smem = (size_t)W * sizeof(float);
    NXD_REQUIRE(smem <= 200 * 1024, "embedding: width %d", W);
    cudaStream_t st = (cudaStream_t)stream;
    constexpr int NT = 256;
#define NXD_EN(TE, TH)                                                                                                   \
    do {                                                                                                                 \
        auto kern = embed_norm_kernel<TE, TH, NT>;                                                                       \
        if (smem > 48 * 1024)                                                                                            \
            NXD_CHECK_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));          \
        kern<<<(unsigned)rows, NT, smem, st>>>((const TE*)table, ids, pos, freq, w_embed, w_next, x, (TH*)h, W, vocab,   \
                                               eps);                                                                     \
    } while (0)
    switch ((e_dtype << 1) | h_dtype) {
        case 0: NXD_EN(bf16, bf16); break;
        case 1: NXD_EN(bf16, float); break;
        case 2: NXD_EN(float, bf16); break;
        default: NXD_EN(float, float);
    }
#undef NXD_EN
    NXD_LAUNCH_CHECK();
    return 0;
}
