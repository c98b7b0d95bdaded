// Flash attention FORWARD on 5th-gen tensor cores (tcgen05 + TMEM + TMA), sm_100a  (SURVEY G4/G6, C23).
//
// Same contract as nxd_flash_attn_fwd in flash_attn.cu (reference: the external NKI `flash_fwd` kernel behind
// src/neuronx_distributed/kernels/flash_attn.py:151-191 and the inference prefill kernel,
// examples/inference/modules/attention/attention_base.py:98-139); this is the fast path, the mma.sync kernel
// stays as the portable fallback and as a second oracle in the tests.
//
// One CTA = 128 query rows of one (batch, head); 192 threads, TWO CTAs per SM so that one CTA's softmax overlaps
// the other CTA's MMAs on the shared tensor core:
//   warp 0    TMA producer: Q once (4-D tensor map over the strided [B,H,S,D] view), then K/V tiles of 64 rows into a
//             3-slot ring in CONSUMPTION order  K0, K1, V0, K2, V1, ...  (so a slot's next load never waits on a
//             late MMA).  K and V tiles have the same smem image (64-wide column groups of 128-byte swizzled rows);
//             only the UMMA descriptor differs: K is the K-major B operand of S = Q K^T, V the MN-major B of O += P V.
//   warp 1    TMEM allocation (O: D columns, S: 64 columns) and MMA issue.  S(j+1) is issued BEFORE waiting for
//             P(j), so it runs while the softmax warps work on tile j.
//   warps 2-5 softmax: one thread per query row (TMEM lane).  tcgen05.ld S -> scale, mask, running max, exp2 ->
//             bf16 P written to tensor memory (tcgen05.st), the A operand of the PV MMA.  O stays in TMEM across the
//             whole loop; it is rescaled (tcgen05.ld / st) only when the running max moved by more than 2^8
//             ("lazy rescale"), which is rare after the first tiles.  Epilogue: O / l -> bf16 -> smem -> TMA store.
#include "common.cuh"
#include "gemm_tcgen05.cuh"
#include "attn_tc_common.cuh"
#include "ptx.cuh"
#include "score_mod.cuh"

#include <type_traits>

namespace {
using namespace nxd_attn;

constexpr int kBM = 128;
constexpr int kBN = 64;
constexpr int kSlots = 3;
constexpr int kThreadsTc = 192;
constexpr float kRescaleThreshold = 8.0f;  // log2 units

struct TcParams {
    float* lse;
    int B, Hq, Hkv, Sq, Sk;
    int pos_q[3], pos_k[3], pos_v[3], pos_o[3];  // coordinate slot (1..3) of (row, head, batch) in each tensor map
    float scale_log2;
    DropParams drop;
    // WIN instantiation only: sliding window with kept first keys and a linear distance bias (causal)
    int window, keep_first;      // window <= 0: no window
    const float* slopes;         // [Hq] or NULL; the bias is -slope * (query position - key position)
    const float* sinks;          // [Hq] or NULL: exp(sink) joins the softmax denominator
    ScoreMod mod;                // output gate; SCORE instantiations: soft cap, logarithmic bias, sigmoid weights
    int bias_entries;            // SCORE: distances in the shared-memory bias table; 0: no bias, -1: evaluated per score
};

template <int D>
struct TcSmem {
    static constexpr int kQBytes = kBM * D * 2;
    static constexpr int kSlotBytes = kBN * D * 2;
    static constexpr int kPBytes = kBM * kBN * 2;
    static constexpr int kQOff = 0;
    static constexpr int kRingOff = kQBytes;
    static constexpr int kPOff = kRingOff + kSlots * kSlotBytes;
    static constexpr int kBarOff = kPOff + kPBytes;
    static constexpr int kNumBars = 1 + 2 * kSlots + 4;
    static constexpr int kBytes = kBarOff + kNumBars * 8 + 16 + 1024;  // + manual 1024-byte alignment slack
    static constexpr int kTmemCols = 256;   // O (D) + S (64) + bf16 P as the tensor-memory A operand of P V (32)
};

// WIN: the key tiles a CTA visits are the ones that hold kept first keys followed by the ones its queries' windows reach
// (`tile(j)` maps the j-th visited tile to its index; every role derives it from the same two numbers), the masked path
// also hides keys below the window that are not kept, and scores get the scale and the distance bias before the running
// max (which is then kept in log2 units).  The barrier protocol and the MMA issue are the same for both instantiations.
// SCORE (with WIN): 1 = soft cap and / or logarithmic distance bias ahead of the softmax, 2 = sigmoid weights (no running max,
// no denominator).  The distance bias of a head is a table over the distances in shared memory, filled once per CTA (lanes are
// query rows, so a warp reads 32 consecutive entries); the soft cap takes the tanh series unless a score of the warp's tile
// is too large for it.
template <int D, bool CAUSAL, bool DROP, bool WIN = false, int SCORE = 0>
__global__ void __launch_bounds__(kThreadsTc, 2)
fa_fwd_tc_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k,
                 const __grid_constant__ CUtensorMap tmap_v, const __grid_constant__ CUtensorMap tmap_o,
                 const TcParams p) {
    using L = TcSmem<D>;
    extern __shared__ __align__(1024) uint8_t smem_raw[];
    uint8_t* smem = align_smem_1024(smem_raw);
    uint8_t* sQ = smem + L::kQOff;
    uint8_t* sRing = smem + L::kRingOff;
    uint8_t* sP = smem + L::kPOff;
    uint64_t* bars = reinterpret_cast<uint64_t*>(smem + L::kBarOff);
    uint64_t* q_full = bars;
    uint64_t* slot_full = bars + 1;
    uint64_t* slot_empty = slot_full + kSlots;
    uint64_t* s_full = slot_empty + kSlots;
    uint64_t* s_empty = s_full + 1;
    uint64_t* p_full = s_empty + 1;
    uint64_t* pv_done = p_full + 1;
    uint32_t* tmem_ptr_smem = reinterpret_cast<uint32_t*>(pv_done + 1);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    // grid = (q heads, batch, q blocks): the q block is the slowest launch dimension and counted from the end, so the
    // long causal rows of EVERY head are scheduled before any short one (longest-first list scheduling)
    const int mb = gridDim.z - 1 - blockIdx.z;
    const int hq = blockIdx.x, b = blockIdx.y;
    const int hkv = hq / (p.Hq / p.Hkv);
    const int m0 = mb * kBM;
    const int offset = p.Sk - p.Sq;
    int n_tiles = (p.Sk + kBN - 1) / kBN;
    if (CAUSAL) n_tiles = min(n_tiles, max((m0 + kBM + offset + kBN - 1) / kBN, 0));
    int n_sink = 0, t_win = 0;
    if (WIN && p.window > 0) {
        t_win = min(max(0, m0 + offset - p.window + 1) / kBN, n_tiles);
        n_sink = min((p.keep_first + kBN - 1) / kBN, t_win);
        n_tiles = n_tiles - t_win + n_sink;
    }
    auto tile = [&](int j) { return WIN ? (j < n_sink ? j : t_win + (j - n_sink)) : j; };

    if (warp == 0 && lane == 0) {
        ptx::prefetch_tensormap(&tmap_q);
        ptx::prefetch_tensormap(&tmap_k);
        ptx::prefetch_tensormap(&tmap_v);
        ptx::prefetch_tensormap(&tmap_o);
        ptx::mbar_init(q_full, 1);
        for (int i = 0; i < kSlots; ++i) {
            ptx::mbar_init(&slot_full[i], 1);
            ptx::mbar_init(&slot_empty[i], 1);
        }
        ptx::mbar_init(s_full, 1);
        ptx::mbar_init(s_empty, 128);
        ptx::mbar_init(p_full, 128);
        ptx::mbar_init(pv_done, 1);
        ptx::fence_barrier_init();
    }
    if (warp == 1) ptx::tmem_alloc<1>(tmem_ptr_smem, L::kTmemCols);
    float* dtab = reinterpret_cast<float*>(sP);          // bias table (SCORE): the P staging area is free, P lives in TMEM
    constexpr float kL2e = score::kLog2e;                // r1 ln(.) in log2 units is r1 log2(.)
    constexpr float kSign = SCORE == 2 ? -1.f : 1.f;     // sigmoid weights are computed from the negative score
    const float r1 = (SCORE > 0 && p.mod.r1 != nullptr) ? p.mod.r1[hq] : 0.f;
    const float r2 = (SCORE > 0 && p.mod.r1 != nullptr) ? p.mod.r2[hq] : 0.f;
    const float bias_slope = (SCORE > 0 && p.slopes != nullptr) ? p.slopes[hq] * kL2e : 0.f;
    const float bias_const = SCORE == 2 ? -p.mod.pb[hq] * kL2e : 0.f;
    // what a score at that distance gains, with the sign of kSign (and the sigmoid's offset)
    auto bias_at = [&](float dist) { return fmaf(-kSign, r1 * __log2f(fmaf(r2, dist, 1.f)) + bias_slope * dist, bias_const); };
    if (SCORE > 0 && p.bias_entries > 0) {
        const int n = min(p.bias_entries, m0 + kBM + offset);
        for (int i = threadIdx.x; i < n; i += kThreadsTc) dtab[i] = bias_at((float)i);
    }
    ptx::tcgen05_fence_before();
    __syncthreads();
    ptx::tcgen05_fence_after();
    const uint32_t tmem_base = *tmem_ptr_smem;
    const uint32_t tmem_o = tmem_base;
    const uint32_t tmem_s = tmem_base + D;
    const uint32_t tmem_p = tmem_base + D + kBN;   // 128 lanes x 64 keys bf16 = 32 packed columns

    if (warp == 0) {
        // ============================ TMA producer ============================
        if (lane == 0 && n_tiles > 0) {
            int c[4];
            ptx::mbar_arrive_expect_tx(q_full, L::kQBytes);
#pragma unroll
            for (int g = 0; g < D / 64; ++g) {
                c[0] = g * 64;
                coords(p.pos_q, m0, hq, b, c);
                tma_load_4d(&tmap_q, q_full, sQ + g * (kBM * 128), c[0], c[1], c[2], c[3]);
            }
            int it = 0;
            auto load = [&](const CUtensorMap* map, const int* pos, int row0) {
                const int slot = it % kSlots;
                const uint32_t ph = (uint32_t)(it / kSlots) & 1u;
                ptx::mbar_wait(&slot_empty[slot], ph ^ 1u);
                ptx::mbar_arrive_expect_tx(&slot_full[slot], L::kSlotBytes);
#pragma unroll
                for (int g = 0; g < D / 64; ++g) {
                    c[0] = g * 64;
                    coords(pos, row0, hkv, b, c);
                    tma_load_4d(map, &slot_full[slot], sRing + slot * L::kSlotBytes + g * (kBN * 128), c[0], c[1], c[2],
                                c[3]);
                }
                ++it;
            };
            load(&tmap_k, p.pos_k, tile(0) * kBN);
            for (int j = 0; j < n_tiles; ++j) {
                if (j + 1 < n_tiles) load(&tmap_k, p.pos_k, tile(j + 1) * kBN);
                load(&tmap_v, p.pos_v, tile(j) * kBN);
            }
        }
    } else if (warp == 1) {
        // ============================ MMA issuer ============================
        if (lane == 0 && n_tiles > 0) {
            constexpr uint32_t idesc_s = ptx::make_idesc_bf16(kBM, kBN, 0, 0);
            constexpr uint32_t idesc_o = ptx::make_idesc_bf16(kBM, D, 0, 1);
            const uint32_t q_addr = ptx::smem_u32(sQ), ring_addr = ptx::smem_u32(sRing);
            int it = 0;
            auto issue_s = [&](int j) {
                const int slot = it % kSlots;
                const uint32_t ph = (uint32_t)(it / kSlots) & 1u;
                ++it;
                ptx::mbar_wait(&slot_full[slot], ph);
                ptx::mbar_wait(s_empty, ((uint32_t)j & 1u) ^ 1u);  // softmax(j-1) has read S out of TMEM
                ptx::tcgen05_fence_after();
                const uint32_t kb = ring_addr + slot * L::kSlotBytes;
#pragma unroll
                for (int kk = 0; kk < D / 16; ++kk) {
                    const uint64_t da = ptx::make_smem_desc(q_addr + (kk >> 2) * (kBM * 128) + (kk & 3) * 32, 16, 1024);
                    const uint64_t db = ptx::make_smem_desc(kb + (kk >> 2) * (kBN * 128) + (kk & 3) * 32, 16, 1024);
                    ptx::umma_bf16<1>(tmem_s, da, db, idesc_s, kk != 0 ? 1u : 0u);
                }
                ptx::umma_commit(&slot_empty[slot]);
                ptx::umma_commit(s_full);
            };
            ptx::mbar_wait(q_full, 0);
            issue_s(0);
            for (int j = 0; j < n_tiles; ++j) {
                if (j + 1 < n_tiles) issue_s(j + 1);
                const int slot = it % kSlots;
                const uint32_t ph = (uint32_t)(it / kSlots) & 1u;
                ++it;
                ptx::mbar_wait(&slot_full[slot], ph);
                ptx::mbar_wait(p_full, (uint32_t)j & 1u);
                ptx::tcgen05_fence_after();
                const uint32_t vb = ring_addr + slot * L::kSlotBytes;
#pragma unroll
                for (int kk = 0; kk < kBN / 16; ++kk) {
                    const uint64_t db = ptx::make_smem_desc(vb + kk * 2048, kBN * 128, 1024);
                    ptx::umma_bf16_ts(tmem_o, tmem_p + kk * 8, db, idesc_o, (j | kk) != 0 ? 1u : 0u);
                }
                ptx::umma_commit(&slot_empty[slot]);
                ptx::umma_commit(pv_done);
            }
        }
    } else {
        // ============================ softmax / epilogue ============================
        const int q = warp & 3;                 // TMEM lane quadrant of this warp
        const int row = q * 32 + lane;          // row inside the q tile == TMEM lane
        const int grow = m0 + row;
        const uint32_t lane_off = (uint32_t)(q * 32) << 16;
        // Running max in RAW score units (the scale is positive, so max commutes with it); the exponent argument is one
        // FFMA per element: s * scale_log2 - m * scale_log2.
        float m_run = -INFINITY, l_run = 0.f;
        const float sc = WIN ? 1.f : p.scale_log2;                   // WIN: scores are converted to log2 units up front
        const float cap_in = (SCORE > 0 && p.mod.cap > 0.f) ? p.scale_log2 / (kL2e * p.mod.cap) : 0.f;
        const float cap_out = kSign * p.mod.cap * kL2e;
        // capped score = s P(s^2): the tanh series with the scales inside (no cap: P is the constant scale)
        const float ci2 = cap_in * cap_in, s_limit = cap_in > 0.f ? score::kSeriesLimit / cap_in : INFINITY;
        const float q0 = kSign * p.scale_log2, q1 = -q0 * ci2 / 3.f, q2 = q0 * ci2 * ci2 * (2.f / 15.f);
        const float q3 = -q0 * ci2 * ci2 * ci2 * (17.f / 315.f), q4 = q0 * ci2 * ci2 * ci2 * ci2 * (62.f / 2835.f);
        const uint64_t k0 = f2_pack(q0, q0), k1 = f2_pack(q1, q1), k2 = f2_pack(q2, q2), k3 = f2_pack(q3, q3), k4 = f2_pack(q4, q4);
        const float slope2 = (WIN && p.slopes != nullptr) ? p.slopes[hq] * 1.4426950408889634f : 0.f;
        // one tile of the online softmax; MASK is instantiated only for tiles on the causal diagonal / past Sk
        auto tile_softmax = [&](auto mask_tag, int j) {
            constexpr bool MASK = decltype(mask_tag)::value;
            uint32_t sr[kBN];
            ptx::tmem_ld_32x32b_x32(tmem_s + lane_off, sr);
            ptx::tmem_ld_32x32b_x32(tmem_s + lane_off + 32, sr + 32);
            ptx::tmem_ld_wait();
            ptx::tcgen05_fence_before();
            ptx::mbar_arrive(s_empty);
            const int n0 = tile(j) * kBN;
            if (SCORE > 0) {
                // sr <- score in log2 units (SCORE 2: its negative), two columns per packed instruction: the capped score is
                // s * P(s^2) with the cap's scales inside P, the bias joins in the last multiply-add
                const int d0 = grow + offset - n0;                          // distance of column 0
                float am0 = 0.f, am1 = 0.f;
#pragma unroll
                for (int c = 0; c < kBN; c += 2) {
                    am0 = fmaxf(am0, fabsf(__uint_as_float(sr[c])));
                    am1 = fmaxf(am1, fabsf(__uint_as_float(sr[c + 1])));
                }
                const bool series = !__any_sync(0xffffffffu, fmaxf(am0, am1) >= s_limit);
                auto cap_and_bias = [&](auto bias) {                        // bias(c): what columns c, c + 1 gain
                    if (series) {
#pragma unroll
                        for (int c = 0; c < kBN; c += 2) {
                            const uint64_t s2 = f2_pack(__uint_as_float(sr[c]), __uint_as_float(sr[c + 1]));
                            const uint64_t z = f2_mul(s2, s2);
                            uint64_t h = f2_fma(z, k4, k3);
                            h = f2_fma(z, h, k2);
                            h = f2_fma(z, h, k1);
                            h = f2_fma(z, h, k0);
                            h = f2_fma(s2, h, bias(c));
                            sr[c] = (uint32_t)h;
                            sr[c + 1] = (uint32_t)(h >> 32);
                        }
                    } else {
#pragma unroll
                        for (int c = 0; c < kBN; c += 2) {
                            const uint64_t t = bias(c);
                            sr[c] = __float_as_uint(fmaf(cap_out, score::tanh_exp(__uint_as_float(sr[c]) * cap_in), f2_lo(t)));
                            sr[c + 1] = __float_as_uint(fmaf(cap_out, score::tanh_exp(__uint_as_float(sr[c + 1]) * cap_in), f2_hi(t)));
                        }
                    }
                };
                if (p.bias_entries > 0) {
                    const float* tb = dtab + d0;
                    if (MASK)
                        cap_and_bias([&](int c) { return f2_pack(dtab[min(max(d0 - c, 0), p.bias_entries - 1)],
                                                                 dtab[min(max(d0 - c - 1, 0), p.bias_entries - 1)]); });
                    else
                        cap_and_bias([&](int c) { return f2_pack(tb[-c], tb[-c - 1]); });
                } else if (p.bias_entries < 0) {
                    cap_and_bias([&](int c) { return f2_pack(bias_at((float)max(d0 - c, 0)), bias_at((float)max(d0 - c - 1, 0))); });
                } else {
                    const uint64_t t = f2_pack(bias_const, bias_const);
                    cap_and_bias([&](int) { return t; });
                }
            } else if (WIN) {
                // log2 units: s * scale - slope * (query position - key position)
                const float base = -slope2 * (float)(grow + offset - n0);
#pragma unroll
                for (int c = 0; c < kBN; ++c)
                    sr[c] = __float_as_uint(fmaf(__uint_as_float(sr[c]), p.scale_log2, fmaf(slope2, (float)c, base)));
            }
            if (MASK) {
                // columns c >= first_bad are masked: beyond the causal diagonal of this row, or beyond the sequence end
                int first_bad = p.Sk - n0;
                if (CAUSAL) first_bad = min(first_bad, grow + offset + 1 - n0);
                // WIN: columns below the window that are not kept first keys are masked as well
                const int first_good = (WIN && p.window > 0) ? grow + offset - p.window + 1 - n0 : 0;
                const int kept = WIN ? p.keep_first - n0 : 0;
#pragma unroll
                for (int c = 0; c < kBN; ++c)
                    if (c >= first_bad || (WIN && c < first_good && c >= kept)) sr[c] = SCORE == 2 ? 0x7f800000u : 0xff800000u;   // -inf
            }
            uint32_t pk[kBN / 2];
            if constexpr (SCORE == 2) {
                // sigmoid(x) = 1 / (1 + 2^-x2), sr = -x2; one reciprocal serves two weights (the clamp keeps the product finite)
#pragma unroll
                for (int c = 0; c < kBN; c += 2) {
                    const float y0 = __uint_as_float(sr[c]), y1 = __uint_as_float(sr[c + 1]);
                    const float a = 1.f + ex2_approx(fminf(y0, 60.f)), bq = 1.f + ex2_approx(fminf(y1, 60.f));
                    const float r = rcp_approx(a * bq);
                    float p0 = r * bq, p1 = r * a;
                    if (MASK) {
                        if (y0 == INFINITY) p0 = 0.f;
                        if (y1 == INFINITY) p1 = 0.f;
                    }
                    pk[c >> 1] = pack_bf16x2(p0, p1);
                }
                l_run = 1.f;
                if (j > 0) {
                    ptx::mbar_wait(pv_done, ((uint32_t)(j - 1)) & 1u);  // P buffer free
                    ptx::tcgen05_fence_after();
                }
            } else {
            float mx0 = __uint_as_float(sr[0]), mx1 = __uint_as_float(sr[1]), mx2 = __uint_as_float(sr[2]),
                  mx3 = __uint_as_float(sr[3]);
#pragma unroll
            for (int c = 4; c < kBN; c += 4) {
                mx0 = fmaxf(mx0, __uint_as_float(sr[c]));
                mx1 = fmaxf(mx1, __uint_as_float(sr[c + 1]));
                mx2 = fmaxf(mx2, __uint_as_float(sr[c + 2]));
                mx3 = fmaxf(mx3, __uint_as_float(sr[c + 3]));
            }
            const float mx = fmaxf(fmaxf(mx0, mx1), fmaxf(mx2, mx3));
            // lazy rescale: keep the stale max unless it moved by more than 2^8 (in scaled log2 units)
            float alpha = 1.f;
            bool rescale = false;
            if ((mx - m_run) * sc > kRescaleThreshold || m_run == -INFINITY) {
                const float m_new = fmaxf(m_run, mx);
                if (m_new != -INFINITY) {
                    alpha = ex2_approx((m_run - m_new) * sc);   // 0 when m_run was -inf
                    rescale = (j > 0) && (m_run != -INFINITY);
                    m_run = m_new;
                }
            }
            const float neg_m = (m_run == -INFINITY) ? 0.f : -m_run * sc;
            float rs0 = 0.f, rs1 = 0.f;
#pragma unroll
            for (int c = 0; c < kBN; c += 2) {
                const float p0 = ex2_approx(fmaf(__uint_as_float(sr[c]), sc, neg_m));
                const float p1 = ex2_approx(fmaf(__uint_as_float(sr[c + 1]), sc, neg_m));
                rs0 += p0;
                rs1 += p1;
                if (DROP) {   // the row sum (softmax denominator) is taken before dropout, the PV operand after it
                    const uint32_t hs = drop_head_seed(p.drop.seed, (uint32_t)(b * p.Hq + hq));
                    const bool k0 = drop_keep(hs, (uint32_t)grow, (uint32_t)(n0 + c), p.drop.threshold);
                    const bool k1 = drop_keep(hs, (uint32_t)grow, (uint32_t)(n0 + c + 1), p.drop.threshold);
                    pk[c >> 1] = pack_bf16x2(k0 ? p0 * p.drop.inv_keep : 0.f, k1 ? p1 * p.drop.inv_keep : 0.f);
                } else {
                    pk[c >> 1] = pack_bf16x2(p0, p1);
                }
            }
            l_run = l_run * alpha + (rs0 + rs1);
            if (j > 0) {
                ptx::mbar_wait(pv_done, ((uint32_t)(j - 1)) & 1u);  // P buffer free, O up to date
                ptx::tcgen05_fence_after();
                if (__any_sync(0xffffffffu, rescale)) {
#pragma unroll 1
                    for (int c = 0; c < D / 32; ++c) {
                        uint32_t o[32];
                        ptx::tmem_ld_32x32b_x32(tmem_o + lane_off + c * 32, o);
                        ptx::tmem_ld_wait();
                        const float a_o = rescale ? alpha : 1.f;
#pragma unroll
                        for (int e = 0; e < 32; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * a_o);
                        tmem_st_32x32b_x32(tmem_o + lane_off + c * 32, o);
                    }
                    tmem_st_wait();
                }
            }
            }
            // P goes to TENSOR MEMORY (this thread's row, 64 keys = 32 packed words): the A operand of the P V MMA never
            // touches shared memory (no 16 KB store + re-read per tile, no async-proxy fence)
            tmem_st_32x32b_x16(tmem_p + lane_off, pk);
            tmem_st_32x32b_x16(tmem_p + lane_off + 16, pk + 16);
            tmem_st_wait();
            ptx::tcgen05_fence_before();
            ptx::mbar_arrive(p_full);
        };
        for (int j = 0; j < n_tiles; ++j) {
            ptx::mbar_wait(s_full, (uint32_t)j & 1u);
            ptx::tcgen05_fence_after();
            const int n0 = tile(j) * kBN;
            // warp-uniform: the tile crosses the sequence end, or the causal diagonal of one of this warp's 32 rows,
            // or (WIN) the lower edge of the window of one of them while not all of it is kept
            const bool need_mask = (n0 + kBN > p.Sk) || (CAUSAL && (n0 + kBN - 1 > m0 + q * 32 + offset)) ||
                                   (WIN && p.window > 0 && m0 + q * 32 + 31 + offset - p.window + 1 > n0 &&
                                    n0 + kBN > p.keep_first);
            if (need_mask) tile_softmax(std::true_type{}, j);
            else tile_softmax(std::false_type{}, j);
        }
        // ---- epilogue ----
        if (n_tiles > 0) {
            ptx::mbar_wait(pv_done, ((uint32_t)(n_tiles - 1)) & 1u);
            ptx::tcgen05_fence_after();
        }
        if (WIN && SCORE != 2 && p.sinks != nullptr && m_run != -INFINITY) l_run += ex2_approx(p.sinks[hq] * kL2e - m_run);
        float inv = l_run > 0.f ? 1.f / l_run : 0.f;
        if (WIN && grow < p.Sq) inv *= score::out_gate<bf16>(p.mod, (long long)b * p.Sq + grow, hq);
        if (p.lse && grow < p.Sq)
            p.lse[((long long)b * p.Hq + hq) * p.Sq + grow] = l_run > 0.f ? m_run * sc + log2f(l_run) : INFINITY;
        // every MMA that read Q has completed: reuse the Q tile as staging (warp q owns rows [32q, 32q+32) of
        // each 64-column group: 32 rows x 128 bytes = one TMA store box)
#pragma unroll 1
        for (int g = 0; g < D / 64; ++g) {
            uint32_t o[64];
            if (n_tiles > 0) {
                ptx::tmem_ld_32x32b_x32(tmem_o + lane_off + g * 64, o);
                ptx::tmem_ld_32x32b_x32(tmem_o + lane_off + g * 64 + 32, o + 32);
                ptx::tmem_ld_wait();
            } else {
#pragma unroll
                for (int e = 0; e < 64; ++e) o[e] = 0u;
            }
            uint8_t* dst = sQ + g * (kBM * 128) + row * 128;
#pragma unroll
            for (int c = 0; c < 8; ++c) {
                uint32_t w[4];
                float eg[8];
                if (WIN && p.mod.gate_cols > 0) {                // one gate number per element
                    const long long at = ((long long)b * p.Sq + min(grow, p.Sq - 1)) * p.mod.gate_ld + (long long)hq * D + g * 64 + c * 8;
                    unpack8(*reinterpret_cast<const bf16x8*>(reinterpret_cast<const bf16*>(p.mod.gate) + at), eg);
#pragma unroll
                    for (int e = 0; e < 8; ++e) eg[e] = p.mod.gate_mul * score::sigmoid(eg[e]) * inv;
                } else {
#pragma unroll
                    for (int e = 0; e < 8; ++e) eg[e] = inv;
                }
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    bf162 t = __floats2bfloat162_rn(__uint_as_float(o[8 * c + 2 * e]) * eg[2 * e],
                                                    __uint_as_float(o[8 * c + 2 * e + 1]) * eg[2 * e + 1]);
                    w[e] = *reinterpret_cast<uint32_t*>(&t);
                }
                st_shared_v4(dst + ((c ^ (row & 7)) << 4), w[0], w[1], w[2], w[3]);
            }
            ptx::fence_proxy_async();
            __syncwarp();
            if (lane == 0 && m0 + q * 32 < p.Sq) {
                int c[4];
                c[0] = g * 64;
                coords(p.pos_o, m0 + q * 32, hq, b, c);
                tma_store_4d(&tmap_o, sQ + g * (kBM * 128) + q * 32 * 128, c[0], c[1], c[2], c[3]);
                ptx::bulk_commit();
            }
        }
        if (lane == 0) ptx::bulk_wait<0>();
    }
    ptx::tcgen05_fence_before();
    __syncthreads();
    if (warp == 1) ptx::tmem_dealloc<1>(tmem_base, L::kTmemCols);
}

template <int D, bool CAUSAL, bool DROP>
int launch_fwd_tc_one(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, const CUtensorMap& to,
                      const TcParams& p, cudaStream_t st) {
    using L = TcSmem<D>;
    dim3 grid(p.Hq, p.B, (p.Sq + kBM - 1) / kBM);
    static cudaError_t once = cudaFuncSetAttribute(fa_fwd_tc_kernel<D, CAUSAL, DROP>,
                                                   cudaFuncAttributeMaxDynamicSharedMemorySize, L::kBytes);
    NXD_CHECK_CUDA(once);
    fa_fwd_tc_kernel<D, CAUSAL, DROP><<<grid, kThreadsTc, L::kBytes, st>>>(tq, tk, tv, to, p);
    NXD_LAUNCH_CHECK();
    return 0;
}

template <int D>
int launch_fwd_tc(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, const CUtensorMap& to,
                  const TcParams& p, int causal, cudaStream_t st) {
    const bool drop = p.drop.threshold != 0;
    if (causal) return drop ? launch_fwd_tc_one<D, true, true>(tq, tk, tv, to, p, st)
                            : launch_fwd_tc_one<D, true, false>(tq, tk, tv, to, p, st);
    return drop ? launch_fwd_tc_one<D, false, true>(tq, tk, tv, to, p, st)
                : launch_fwd_tc_one<D, false, false>(tq, tk, tv, to, p, st);
}

template <int D, int SCORE>
int launch_fwd_tc_win(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, const CUtensorMap& to,
                      const TcParams& p, cudaStream_t st) {
    using L = TcSmem<D>;
    dim3 grid(p.Hq, p.B, (p.Sq + kBM - 1) / kBM);
    static cudaError_t once = cudaFuncSetAttribute(fa_fwd_tc_kernel<D, true, false, true, SCORE>,
                                                   cudaFuncAttributeMaxDynamicSharedMemorySize, L::kBytes);
    NXD_CHECK_CUDA(once);
    fa_fwd_tc_kernel<D, true, false, true, SCORE><<<grid, kThreadsTc, L::kBytes, st>>>(tq, tk, tv, to, p);
    NXD_LAUNCH_CHECK();
    return 0;
}

}  // namespace

// Same arguments as nxd_flash_attn_fwd.  Extra requirement: 16-byte aligned base pointers.
static int fwd_tc_impl(const void* q, const void* k, const void* v, void* o, float* lse, const long long* strides, int B,
                       int Hq, int Hkv, int Sq, int Sk, int D, float scale, int causal, float dropout_p,
                       unsigned long long seed, void* stream) {
    NXD_REQUIRE(D == 64 || D == 128, "flash_attn_tc: head dim %d not supported (64 or 128)", D);
    NXD_REQUIRE(B > 0 && Hq > 0 && Hkv > 0 && Sq > 0 && Sk > 0 && Hq % Hkv == 0, "flash_attn_tc: bad problem");
    for (int i = 0; i < 12; ++i)
        NXD_REQUIRE(strides[i] % 8 == 0, "flash_attn_tc: stride %d (=%lld) must be a multiple of 8 elements", i,
                    strides[i]);
    NXD_REQUIRE((((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)o) & 15) == 0,
                "flash_attn_tc: tensors must be 16-byte aligned");
    TcParams p{};
    p.lse = lse;
    p.B = B; p.Hq = Hq; p.Hkv = Hkv; p.Sq = Sq; p.Sk = Sk;
    p.scale_log2 = scale * 1.4426950408889634f;
    NXD_REQUIRE(dropout_p >= 0.f && dropout_p < 1.f, "flash_attn_tc: dropout_p %f not in [0, 1)", dropout_p);
    p.drop.threshold = dropout_p > 0.f ? (uint32_t)fmin(4294967295.0, (double)dropout_p * 4294967296.0) : 0u;
    p.drop.inv_keep = 1.f / (1.f - dropout_p);
    p.drop.seed = (uint32_t)(seed ^ (seed >> 32));
    CUtensorMap tq, tk, tv, to;
    int rc;
    if ((rc = make_tmap_bhsd(&tq, q, D, Sq, Hq, B, strides[2], strides[1], strides[0], kBM, p.pos_q))) return rc;
    if ((rc = make_tmap_bhsd(&tk, k, D, Sk, Hkv, B, strides[5], strides[4], strides[3], kBN, p.pos_k))) return rc;
    if ((rc = make_tmap_bhsd(&tv, v, D, Sk, Hkv, B, strides[8], strides[7], strides[6], kBN, p.pos_v))) return rc;
    if ((rc = make_tmap_bhsd(&to, o, D, Sq, Hq, B, strides[11], strides[10], strides[9], 32, p.pos_o))) return rc;
    return D == 64 ? launch_fwd_tc<64>(tq, tk, tv, to, p, causal, (cudaStream_t)stream)
                   : launch_fwd_tc<128>(tq, tk, tv, to, p, causal, (cudaStream_t)stream);
}

NXD_API int nxd_flash_attn_fwd_tc(const void* q, const void* k, const void* v, void* o, float* lse,
                                  const long long* strides, int B, int Hq, int Hkv, int Sq, int Sk, int D, float scale,
                                  int causal, void* stream) {
    return fwd_tc_impl(q, k, v, o, lse, strides, B, Hq, Hkv, Sq, Sk, D, scale, causal, 0.f, 0ull, stream);
}

// Same, with attention dropout: P is multiplied by a keep mask / (1 - dropout_p) before the PV product; the mask is a
// function of (seed, batch, head, query, key) that nxd_flash_attn_bwd_tc_dropout regenerates.
NXD_API int nxd_flash_attn_fwd_tc_dropout(const void* q, const void* k, const void* v, void* o, float* lse,
                                          const long long* strides, int B, int Hq, int Hkv, int Sq, int Sk, int D,
                                          float scale, int causal, float dropout_p, unsigned long long seed,
                                          void* stream) {
    return fwd_tc_impl(q, k, v, o, lse, strides, B, Hq, Hkv, Sq, Sk, D, scale, causal, dropout_p, seed, stream);
}

// Causal attention with a sliding window (window <= 0: none), `keep_first` first keys that stay visible, and a linear
// distance bias -slopes[h] * (i - j) (slopes NULL: none); tensors and strides as nxd_flash_attn_fwd_tc, no lse output.
// sinks [Hq] or NULL; softcap, log_r1 / log_r2, sigmoid_bias, gate as in nxd_scored_attn_prefill (score_mod.cuh).
NXD_API int nxd_flash_attn_fwd_tc_scored(const void* q, const void* k, const void* v, void* o, const long long* strides,
                                         int B, int Hq, int Hkv, int Sq, int Sk, int D, float scale, int window,
                                         int keep_first, const float* slopes, const float* sinks, float softcap,
                                         const float* log_r1, const float* log_r2, const float* sigmoid_bias,
                                         const void* gate, long long gate_ld, int gate_cols, float gate_mul, void* stream) {
    NXD_REQUIRE(gate_cols == 0 || (gate_cols == D && gate != nullptr && gate_ld % 8 == 0 && ((uintptr_t)gate & 15) == 0),
                "flash_attn_tc: a gate of %d columns per head of %d", gate_cols, D);
    NXD_REQUIRE((log_r1 == nullptr) == (log_r2 == nullptr), "flash_attn_tc: the logarithmic bias needs %s", "both vectors");
    NXD_REQUIRE(sigmoid_bias == nullptr || sinks == nullptr, "flash_attn_tc: sigmoid weights have no %s", "sink");
    NXD_REQUIRE(D == 64 || D == 128, "flash_attn_tc_window: head dim %d not supported (64 or 128)", D);
    NXD_REQUIRE(B > 0 && Hq > 0 && Hkv > 0 && Sq > 0 && Sk >= Sq && Hq % Hkv == 0, "flash_attn_tc_window: bad problem");
    for (int i = 0; i < 12; ++i)
        NXD_REQUIRE(strides[i] % 8 == 0, "flash_attn_tc_window: stride %d (=%lld) must be a multiple of 8 elements", i,
                    strides[i]);
    NXD_REQUIRE((((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)o) & 15) == 0,
                "flash_attn_tc_window: tensors must be 16-byte aligned");
    TcParams p{};
    p.lse = nullptr;
    p.B = B; p.Hq = Hq; p.Hkv = Hkv; p.Sq = Sq; p.Sk = Sk;
    p.scale_log2 = scale * 1.4426950408889634f;
    p.drop.threshold = 0u;
    p.drop.inv_keep = 1.f;
    p.window = window;
    p.keep_first = keep_first > 0 ? keep_first : 0;
    p.slopes = slopes;
    p.sinks = sinks;
    p.mod = ScoreMod{softcap > 0.f ? softcap : 0.f, log_r1, log_r2, sigmoid_bias, gate, gate_ld, gate_cols, gate_mul, 0};
    const int mode = p.mod.mode();
    if (mode > 0 && (log_r1 != nullptr || slopes != nullptr)) {
        const int span = (window > 0 && window < Sk && p.keep_first == 0) ? window : Sk;      // distances that can be visible
        p.bias_entries = span <= TcSmem<64>::kPBytes / 4 ? span : -1;
    }
    CUtensorMap tq, tk, tv, to;
    int rc;
    if ((rc = make_tmap_bhsd(&tq, q, D, Sq, Hq, B, strides[2], strides[1], strides[0], kBM, p.pos_q))) return rc;
    if ((rc = make_tmap_bhsd(&tk, k, D, Sk, Hkv, B, strides[5], strides[4], strides[3], kBN, p.pos_k))) return rc;
    if ((rc = make_tmap_bhsd(&tv, v, D, Sk, Hkv, B, strides[8], strides[7], strides[6], kBN, p.pos_v))) return rc;
    if ((rc = make_tmap_bhsd(&to, o, D, Sq, Hq, B, strides[11], strides[10], strides[9], 32, p.pos_o))) return rc;
    cudaStream_t st = (cudaStream_t)stream;
    if (mode == 2) return D == 64 ? launch_fwd_tc_win<64, 2>(tq, tk, tv, to, p, st) : launch_fwd_tc_win<128, 2>(tq, tk, tv, to, p, st);
    if (mode == 1) return D == 64 ? launch_fwd_tc_win<64, 1>(tq, tk, tv, to, p, st) : launch_fwd_tc_win<128, 1>(tq, tk, tv, to, p, st);
    return D == 64 ? launch_fwd_tc_win<64, 0>(tq, tk, tv, to, p, st) : launch_fwd_tc_win<128, 0>(tq, tk, tv, to, p, st);
}

NXD_API int nxd_flash_attn_fwd_tc_window(const void* q, const void* k, const void* v, void* o, const long long* strides,
                                         int B, int Hq, int Hkv, int Sq, int Sk, int D, float scale, int window,
                                         int keep_first, const float* slopes, void* stream) {
    return nxd_flash_attn_fwd_tc_scored(q, k, v, o, strides, B, Hq, Hkv, Sq, Sk, D, scale, window, keep_first, slopes, nullptr,
                                        0.f, nullptr, nullptr, nullptr, nullptr, 0, 0, 1.f, stream);
}
