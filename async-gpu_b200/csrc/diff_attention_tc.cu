// Differential attention of prompt rows on the tensor cores (tcgen05, accumulators in tensor memory), bfloat16.
//
// One block per (128-query tile, head, sequence), ten warps; both softmax maps of a head run side by side over the
// same value tiles, so that one map's softmax covers the other's matrix products:
//   warp 0      copies: the query tile of both maps once, then 128-key tiles of the cache (keys of both maps, values)
//   warp 1      MMA issue: S_m = Q_m K_m^T for map m, O_m += P_m V with P read from tensor memory and V straight from
//               its row-major tile
//   warps 2..5  softmax of map 0, one query row per thread; warps 6..9 of map 1
// At the end the threads of map 0 hold a row of both outputs: o = O_0 / l_0 - lambda O_1 / l_1 in f32, over its root
// mean square, times (1 - diff) and the head's gate.
//
// TMEM (512 columns, one block per SM): scores of map m at columns 256 m (P overwrites the first 64 as packed pairs),
// O_m at 256 m + 128.  O_m stays there over the key tiles; the reference maximum moves (and O_m is rescaled) only when a
// score exceeds it by more than 2^8.
//
// Scores s = q . k times scale and the row's temperature pass cap * tanh(s / cap).  While a row's |s / cap| stay within
// 1/2 in a tile the tangent is an odd polynomial (fitted to tanh on that interval, relative error 3e-8), otherwise
// 1 - 2 / (1 + e^2x).
//
// Every mbarrier wait is bounded (see attention_tc.cu).
#include <cuda.h>

#include <algorithm>

#include "device_utils.cuh"
#include "hybrid.h"
#include "tc_ptx.cuh"

namespace {

constexpr float NEG_BIG = -1.0e30f, LOG2E = 1.4426950408889634f;
enum : uint32_t { ERR_DP_Q = 0x81, ERR_DP_K, ERR_DP_V, ERR_DP_S, ERR_DP_P, ERR_DP_O, ERR_DP_KE, ERR_DP_VE };
constexpr int TM_COLS = 512;
constexpr int BOX = 16384; // 128 rows x 64 bf16
constexpr int NTHREADS = 320;

struct Bars {
    uint64_t q_full, done;
    uint64_t k_full[2], k_empty[2], v_full[2], v_empty[2];
    uint64_t s_full[2], p_full[2]; // per map
};

__device__ __forceinline__ float rcp_approx(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// KB: 64-column boxes of a map's key; VB: of a value; VS: value stages; CAP: scores are capped.
template <int KB, int VB, int VS, bool CAP>
__global__ void __launch_bounds__(NTHREADS, 1)
diff_prefill_tc_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_c, DiffDims d, int cap_rows, SeqMap sm,
                       const float *__restrict__ gate, int gate_ld, __nv_bfloat16 *__restrict__ out, uint32_t *__restrict__ dev_err) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ __align__(8) Bars bars;
    __shared__ float row_sum[128]; // of map 1
    __shared__ uint32_t tmem_slot;
    __shared__ int abort_flag;

    // the query tiles with the most key tiles are scheduled first
    const int h = blockIdx.x, sidx = blockIdx.y, qt = gridDim.z - 1 - blockIdx.z;
    const int tid = threadIdx.x, warp = tid >> 5;
    pdl_wait();
    const int n = sm.n[sidx];
    if (qt * 128 >= n) return; // the whole block
    const uint32_t base = (tc::smem_u32(smem_raw) + 1023u) & ~1023u;
    const uint32_t sQ = base, sK = sQ + 2 * KB * BOX, sV = sK + 4 * KB * BOX;
    auto bar = [&](const uint64_t &x) { return tc::smem_u32(&x); };

    if (tid == 0) {
        abort_flag = 0;
        tc::mbar_init(bar(bars.q_full), 1);
        tc::mbar_init(bar(bars.done), 1);
        for (int i = 0; i < 2; ++i) {
            tc::mbar_init(bar(bars.k_full[i]), 1);
            tc::mbar_init(bar(bars.k_empty[i]), 1);
            tc::mbar_init(bar(bars.v_full[i]), 1);
            tc::mbar_init(bar(bars.v_empty[i]), 1);
            tc::mbar_init(bar(bars.s_full[i]), 1);
            tc::mbar_init(bar(bars.p_full[i]), 128); // every softmax thread of the map
        }
        tc::fence_mbar_init();
    }
    if (warp == 1) tc::tmem_alloc(tc::smem_u32(&tmem_slot), TM_COLS);
    tc::tc_fence_before_sync();
    __syncthreads();
    tc::tc_fence_after_sync();
    pdl_trigger(); // only now: a dependent block must not take this one's tensor memory
    const uint32_t tmem_base = *reinterpret_cast<volatile uint32_t *>(&tmem_slot);

    const int past = sm.past[sidx], row0 = sm.row0[sidx];
    const int kend = past + min(n, qt * 128 + 128); // keys the tile's last row sees
    const int n_tiles = (kend + 127) >> 7;
    const int crow = (sm.slot[sidx] * d.kv_heads + h / d.group()) * cap_rows; // cache row of position 0

    if (warp == 0) {
        // ---- copies: keys one tile ahead of the values ----
        if (tc::elect_one()) {
            tc::mbar_expect_tx(bar(bars.q_full), 2 * KB * BOX);
#pragma unroll
            for (int i = 0; i < 2 * KB; ++i) tc::tma_load_3d(sQ + i * BOX, &tm_q, (i % KB) * 64, 2 * h + i / KB, row0 + qt * 128, bar(bars.q_full));
        }
        __syncwarp();
        auto load_k = [&](int j) {
            const int st = j & 1;
            if (j >= 2 && !tc::mbar_wait(bar(bars.k_empty[st]), ((j >> 1) - 1) & 1, &abort_flag, dev_err, ERR_DP_KE)) return false;
            if (tc::elect_one()) {
                tc::mbar_expect_tx(bar(bars.k_full[st]), 2 * KB * BOX);
#pragma unroll
                for (int i = 0; i < 2 * KB; ++i)
                    tc::tma_load_2d(sK + (st * 2 * KB + i) * BOX, &tm_c, (i / KB) * d.dim_p + (i % KB) * 64, crow + j * 128, bar(bars.k_full[st]));
            }
            __syncwarp();
            return true;
        };
        bool ok = load_k(0);
        for (int j = 0; ok && j < n_tiles; ++j) {
            if (j + 1 < n_tiles) ok = load_k(j + 1);
            if (!ok) break;
            const int st = j % VS;
            if (j >= VS) ok = tc::mbar_wait(bar(bars.v_empty[st]), (j / VS - 1) & 1, &abort_flag, dev_err, ERR_DP_VE);
            if (!ok) break;
            if (tc::elect_one()) {
                tc::mbar_expect_tx(bar(bars.v_full[st]), VB * BOX);
#pragma unroll
                for (int i = 0; i < VB; ++i) tc::tma_load_2d(sV + (st * VB + i) * BOX, &tm_c, 2 * d.dim_p + i * 64, crow + j * 128, bar(bars.v_full[st]));
            }
            __syncwarp();
        }
    } else if (warp == 1) {
        // ---- MMA issue: S of both maps, then per tile and map O_m and the next S_m ----
        constexpr uint32_t idesc_s = tc::umma_idesc_f16(128, 128) | tc::UMMA_BF16;
        constexpr uint32_t idesc_o = tc::umma_idesc_f16_bmn(128, 64) | tc::UMMA_BF16;
        const int steps = d.dim_p >> 4;
        const uint64_t dq = tc::umma_desc_sw128(sQ);
        auto issue_s = [&](int m, int j) { // one elected thread
            const uint64_t off_m = (uint64_t)(m * KB * (BOX >> 4)), dk = tc::umma_desc_sw128(sK + (j & 1) * 2 * KB * BOX) + off_m;
            for (int k = 0; k < steps; ++k) { // 16 columns a step, four steps a box
                const uint64_t off = (uint64_t)((k >> 2) * (BOX >> 4) + (k & 3) * 2);
                tc::umma_f16_ss(tmem_base + 256 * m, dq + off_m + off, dk + off, idesc_s, k != 0);
            }
            tc::umma_commit(bar(bars.s_full[m]));
            if (m) tc::umma_commit(bar(bars.k_empty[j & 1]));
        };
        bool ok = tc::mbar_wait(bar(bars.q_full), 0, &abort_flag, dev_err, ERR_DP_Q);
        if (ok) ok = tc::mbar_wait(bar(bars.k_full[0]), 0, &abort_flag, dev_err, ERR_DP_K);
        if (ok) {
            tc::tc_fence_after_sync();
            if (tc::elect_one()) {
                issue_s(0, 0);
                issue_s(1, 0);
            }
            __syncwarp();
        }
        for (int j = 0; ok && j < n_tiles; ++j) {
            const bool more = j + 1 < n_tiles;
            const int st = j % VS;
            ok = tc::mbar_wait(bar(bars.v_full[st]), (j / VS) & 1, &abort_flag, dev_err, ERR_DP_V);
            if (ok && more) ok = tc::mbar_wait(bar(bars.k_full[(j + 1) & 1]), ((j + 1) >> 1) & 1, &abort_flag, dev_err, ERR_DP_K);
            for (int m = 0; ok && m < 2; ++m) {
                ok = tc::mbar_wait(bar(bars.p_full[m]), j & 1, &abort_flag, dev_err, ERR_DP_P);
                if (!ok) break;
                tc::tc_fence_after_sync();
                if (tc::elect_one()) {
#pragma unroll
                    for (int i = 0; i < VB; ++i) {
                        const uint64_t dv = tc::umma_desc_sw128_mn64(sV + (st * VB + i) * BOX);
#pragma unroll
                        for (int k = 0; k < 8; ++k) // 16 keys per MMA: 8 TMEM columns of P, 2048 bytes of V
                            tc::umma_f16_ts(tmem_base + 256 * m + 128 + i * 64, tmem_base + 256 * m + 8 * k, dv + (uint64_t)(k * (2048 >> 4)), idesc_o,
                                            (j | k) != 0);
                    }
                    if (m) tc::umma_commit(bar(bars.v_empty[st]));
                    if (more) issue_s(m, j + 1);
                    else if (m) tc::umma_commit(bar(bars.done));
                }
                __syncwarp();
            }
        }
    } else {
        // ---- softmax: thread = query row = TMEM lane, map = warpgroup ----
        const int map = (warp - 2) >> 2, quad = warp & 3, row = quad * 32 + (tid & 31);
        const uint32_t lanes = tmem_base + ((uint32_t)(quad * 32) << 16), sbuf = lanes + 256 * map, obuf = sbuf + 128;
        const int s_row = qt * 128 + row;
        const bool row_valid = s_row < n;
        const int pos = past + s_row;
        // scores in units of log2: without a cap s * f, with it cap log2(e) tanh(s * f)
        const float f = CAP ? d.score_scale(pos) / d.cap : d.score_scale(pos) * LOG2E, fc = d.cap * LOG2E;
        auto score = [&](float s) {
            if (!CAP) return s * f;
            return fc * fmaf(-2.0f, rcp_approx(1.0f + tc::ex2_approx(s * f * (2.0f * LOG2E))), 1.0f);
        };
        float m = NEG_BIG, l = 0.0f;
        bool ok = true;
        for (int j = 0; j < n_tiles; ++j) {
            ok = tc::mbar_wait(bar(bars.s_full[map]), j & 1, &abort_flag, dev_err, ERR_DP_S);
            if (!ok) break;
            tc::tc_fence_after_sync();
            const int c1 = row_valid ? min(128, pos + 1 - j * 128) : 0; // columns of the tile the row sees (may be <= 0)
            const bool full = __all_sync(0xffffffffu, c1 == 128);
            // pass 1: largest score and largest magnitude
            float mx[4] = {NEG_BIG, NEG_BIG, NEG_BIG, NEG_BIG}, ma[2] = {0.0f, 0.0f};
#pragma unroll 1
            for (int hf = 0; hf < 2; ++hf) {
                uint32_t v[64];
                tc::tmem_ld_x64(sbuf + 64 * hf, v);
                if (!full)
#pragma unroll
                    for (int e = 0; e < 64; ++e)
                        if (64 * hf + e >= c1) v[e] = __float_as_uint(NEG_BIG);
#pragma unroll
                for (int e = 0; e < 64; e += 8) {
                    mx[0] = tc::fmax3(mx[0], __uint_as_float(v[e]), __uint_as_float(v[e + 1]));
                    mx[1] = tc::fmax3(mx[1], __uint_as_float(v[e + 2]), __uint_as_float(v[e + 3]));
                    mx[2] = tc::fmax3(mx[2], __uint_as_float(v[e + 4]), __uint_as_float(v[e + 5]));
                    mx[3] = tc::fmax3(mx[3], __uint_as_float(v[e + 6]), __uint_as_float(v[e + 7]));
                }
                if (CAP)
#pragma unroll
                    for (int e = 0; e < 64; e += 4) {
                        ma[0] = tc::fmax3(ma[0], fabsf(__uint_as_float(v[e])), fabsf(__uint_as_float(v[e + 1])));
                        ma[1] = tc::fmax3(ma[1], fabsf(__uint_as_float(v[e + 2])), fabsf(__uint_as_float(v[e + 3])));
                    }
            }
            const float top = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3]));
            const float sc = top > NEG_BIG ? score(top) : NEG_BIG;
            // (masked entries count as huge magnitudes: tiles on the diagonal take the general form)
            const bool small = CAP && __all_sync(0xffffffffu, fmaxf(ma[0], ma[1]) * fabsf(f) <= 0.5f);
            if (__any_sync(0xffffffffu, sc > m + 8.0f)) {
                const float m_new = fmaxf(m, sc), corr = tc::ex2_approx(m - m_new);
                if (j > 0) { // the products of the tiles before have retired: this tile's S was issued after them
#pragma unroll 1
                    for (int c = 0; c < 64 * VB; c += 32) {
                        uint32_t o0[16], o1[16];
                        tc::tmem_ld_x16(obuf + c, o0);
                        tc::tmem_ld_x16(obuf + c + 16, o1);
#pragma unroll
                        for (int e = 0; e < 16; ++e) {
                            o0[e] = __float_as_uint(__uint_as_float(o0[e]) * corr);
                            o1[e] = __float_as_uint(__uint_as_float(o1[e]) * corr);
                        }
                        tc::tmem_st_x16(obuf + c, o0);
                        tc::tmem_st_x16(obuf + c + 16, o1);
                    }
                }
                l *= corr;
                m = m_new;
            }
            float ls[4] = {0.0f, 0.0f, 0.0f, 0.0f};
            const uint64_t f2 = f32x2(f, f), nm2 = f32x2(-m, -m);
            // fc times the polynomial's coefficients
            const uint64_t c0 = f32x2(fc, fc), c3 = f32x2(fc * -0.3333307206630707f, fc * -0.3333307206630707f),
                           c5 = f32x2(fc * 0.13324828445911407f, fc * 0.13324828445911407f),
                           c7 = f32x2(fc * -0.05298924073576927f, fc * -0.05298924073576927f),
                           c9 = f32x2(fc * 0.017141319811344147f, fc * 0.017141319811344147f);
#pragma unroll 1
            for (int hf = 0; hf < 2; ++hf) { // pass 2: p = 2^(score - max) as bf16 pairs over the scores
                uint32_t v[64], o[32];
                tc::tmem_ld_x64(sbuf + 64 * hf, v);
                if (!CAP || small) {
#pragma unroll
                    for (int e = 0; e < 64; e += 2) {
                        const uint64_t s2 = f32x2(__uint_as_float(v[e]), __uint_as_float(v[e + 1]));
                        uint64_t e2;
                        if (CAP) {
                            const uint64_t x = mul2(s2, f2), z = mul2(x, x);
                            e2 = fma2(x, fma2(z, fma2(z, fma2(z, fma2(z, c9, c7), c5), c3), c0), nm2);
                        } else {
                            e2 = fma2(s2, f2, nm2);
                        }
                        const float2 ee = f32x2_parts(e2);
                        float p0 = tc::ex2_approx(ee.x), p1 = tc::ex2_approx(ee.y);
                        if (!full) {
                            if (64 * hf + e >= c1) p0 = 0.0f;
                            if (64 * hf + e + 1 >= c1) p1 = 0.0f;
                        }
                        ls[(e >> 1) & 3] += p0 + p1;
                        o[e >> 1] = pack_bf16x2(p0, p1);
                    }
                } else {
#pragma unroll
                    for (int e = 0; e < 64; e += 2) {
                        float p0 = tc::ex2_approx(score(__uint_as_float(v[e])) - m), p1 = tc::ex2_approx(score(__uint_as_float(v[e + 1])) - m);
                        if (!full) {
                            if (64 * hf + e >= c1) p0 = 0.0f;
                            if (64 * hf + e + 1 >= c1) p1 = 0.0f;
                        }
                        ls[(e >> 1) & 3] += p0 + p1;
                        o[e >> 1] = pack_bf16x2(p0, p1);
                    }
                }
                tc::tmem_st_x32(sbuf + 32 * hf, o);
            }
            tc::tmem_st_wait();
            tc::tc_fence_before_sync();
            tc::mbar_arrive(bar(bars.p_full[map]));
            l += (ls[0] + ls[1]) + (ls[2] + ls[3]);
        }
        if (map == 1) row_sum[row] = l;
        asm volatile("bar.sync 1, 256;" ::: "memory");
        if (map == 0 && ok) ok = tc::mbar_wait(bar(bars.done), 0, &abort_flag, dev_err, ERR_DP_O);
        if (map == 0 && ok) {
            tc::tc_fence_after_sync();
            const float f0 = 1.0f / l, f1 = -d.lambda / row_sum[row];
            float acc[64 * VB], ss = 0.0f;
#pragma unroll
            for (int c = 0; c < 64 * VB; c += 16) { // columns past vdim are zero
                uint32_t a[16], b[16];
                tc::tmem_ld_x16(obuf + c, a);
                tc::tmem_ld_x16(obuf + 256 + c, b);
#pragma unroll
                for (int e = 0; e < 16; ++e) {
                    acc[c + e] = fmaf(__uint_as_float(b[e]), f1, __uint_as_float(a[e]) * f0);
                    ss = fmaf(acc[c + e], acc[c + e], ss);
                }
            }
            if (row_valid) {
                const size_t r = row0 + s_row;
                const float g = (1.0f - d.diff) * sigmoid_f(gate[r * gate_ld + h]) / sqrtf(ss / (float)d.vdim + d.eps);
                uint4 *dst = reinterpret_cast<uint4 *>(out + (r * d.heads + h) * d.vdim_p);
#pragma unroll
                for (int c = 0; c < 8 * VB; ++c) {
                    if (8 * c >= d.vdim_p) break;
                    dst[c] = make_uint4(pack_bf16x2(acc[8 * c] * g, acc[8 * c + 1] * g), pack_bf16x2(acc[8 * c + 2] * g, acc[8 * c + 3] * g),
                                        pack_bf16x2(acc[8 * c + 4] * g, acc[8 * c + 5] * g), pack_bf16x2(acc[8 * c + 6] * g, acc[8 * c + 7] * g));
                }
            }
        }
    }

    // ---- teardown (also the path taken after a wait gave up) ----
    if (abort_flag && warp == 0) { // let copies still in flight land before the block's memory is released
        for (int i = 0; i < 64; ++i) __nanosleep(1000);
    }
    tc::tc_fence_before_sync();
    __syncthreads();
    if (warp == 1) tc::tmem_dealloc(tmem_base, TM_COLS);
}

typedef CUresult (*EncodeTiledFn)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *, const cuuint64_t *,
                                  const cuuint64_t *, const cuuint32_t *, const cuuint32_t *, CUtensorMapInterleave,
                                  CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

int encode(b200nn_ctx *ctx, const void *p, int rank, const cuuint64_t *dim, const cuuint64_t *stride, const cuuint32_t *box, CUtensorMap *out) {
    const cuuint32_t ones[3] = {1, 1, 1};
    CUresult r = ((EncodeTiledFn)ctx->encode_tiled)(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, rank, (void *)p, dim, stride, box, ones,
                                                    CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
                                                    CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) return set_error(ctx, B200NN_ERR_CUDA, "cuTensorMapEncodeTiled (differential attention) failed: " + std::to_string((int)r));
    return B200NN_OK;
}

template <int KB, int VB, bool CAP>
int launch_kv(b200nn_ctx *ctx, const DiffDims &d, const CUtensorMap &tq, const CUtensorMap &tcm, int cap, const SeqMap &sm, const float *gate, int gate_ld,
              __nv_bfloat16 *out) {
    constexpr int VS = KB == 2 && VB == 2 ? 1 : 2;
    constexpr int smem = (6 * KB + VS * VB) * BOX + 1024;
    static_assert(smem <= 227 * 1024 - 1024, "shared memory budget exceeded");
    auto kern = diff_prefill_tc_kernel<KB, VB, VS, CAP>;
    static bool attr_done[16] = {};
    if (!attr_done[ctx->device & 15]) {
        CK(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
        prefer_max_smem(kern);
        attr_done[ctx->device & 15] = true;
    }
    const dim3 grid(d.heads, sm.n_seq, (sm.max_n + 127) / 128);
    CK(ctx, launch_pdl(ctx, kern, grid, dim3(NTHREADS), (size_t)smem, tq, tcm, d, cap, sm, gate, gate_ld, out, ctx->dev_err));
    CK_LAUNCH(ctx, "diff_prefill_tc_kernel");
    return B200NN_OK;
}

template <bool CAP>
int launch_cap(b200nn_ctx *ctx, const DiffDims &d, const CUtensorMap &tq, const CUtensorMap &tcm, int cap, const SeqMap &sm, const float *gate, int gate_ld,
               __nv_bfloat16 *out) {
    if (d.dim_p <= 64)
        return d.vdim_p <= 64 ? launch_kv<1, 1, CAP>(ctx, d, tq, tcm, cap, sm, gate, gate_ld, out)
                              : launch_kv<1, 2, CAP>(ctx, d, tq, tcm, cap, sm, gate, gate_ld, out);
    return d.vdim_p <= 64 ? launch_kv<2, 1, CAP>(ctx, d, tq, tcm, cap, sm, gate, gate_ld, out)
                          : launch_kv<2, 2, CAP>(ctx, d, tq, tcm, cap, sm, gate, gate_ld, out);
}

}  // namespace

bool diff_prefill_tc_supported(const b200nn_ctx *ctx, const DiffDims &d) {
    return ctx->attn_tc && ctx->encode_tiled && d.dim_p <= 128 && d.vdim_p <= 128;
}

int launch_diff_prefill_tc(b200nn_ctx *ctx, const DiffDims &d, const __nv_bfloat16 *q, int ldq, const __nv_bfloat16 *cache, int cap, size_t cache_rows,
                           const SeqMap &sm, int n_rows, const float *gate, int gate_ld, __nv_bfloat16 *out) {
    if (sm.n_seq > 65535 || (sm.max_n + 127) / 128 > 65535)
        return set_error(ctx, B200NN_ERR_SHAPE, "differential attention: more than 65535 sequences or query tiles");
    if (cache_rows > 0x7fffffff) return set_error(ctx, B200NN_ERR_SHAPE, "differential attention: more than 2^31 cache rows");
    CUtensorMap tq, tcm;
    { // [n_rows][2 heads][dim_p]
        const cuuint64_t dim[3] = {(cuuint64_t)d.dim_p, (cuuint64_t)2 * d.heads, (cuuint64_t)n_rows}, stride[2] = {(cuuint64_t)d.dim_p * 2, (cuuint64_t)ldq * 2};
        const cuuint32_t box[3] = {64, 1, 128};
        TRY(encode(ctx, q, 3, dim, stride, box, &tq));
    }
    { // [cache_rows][kv_w]
        const cuuint64_t dim[2] = {(cuuint64_t)d.kv_w(), (cuuint64_t)cache_rows}, stride[1] = {(cuuint64_t)d.kv_w() * 2};
        const cuuint32_t box[2] = {64, 128};
        TRY(encode(ctx, cache, 2, dim, stride, box, &tcm));
    }
    return d.cap > 0.0f ? launch_cap<true>(ctx, d, tq, tcm, cap, sm, gate, gate_ld, out) : launch_cap<false>(ctx, d, tq, tcm, cap, sm, gate, gate_ld, out);
}
