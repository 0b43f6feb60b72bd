// Latent attention of prompt rows on the tensor cores (tcgen05, accumulators in tensor memory), bfloat16.
//
// One block per (128-query tile, head, sequence), six warps with the roles of attention_tc.cu: warp 0 copies the
// query tile once and the key and value tiles of every 128-key step through tensor maps into two-stage rings;
// warp 1 issues S = Q K^T, then O = P V with P read from tensor memory and V straight from its row-major tile;
// warps 2..5 are the softmax, one query row per thread.  What differs from attention_tc.cu: a key is two pieces
// (the head's own expanded columns, and the rotated columns all heads share, from the gathered cache rows),
// values may be two 64-column boxes, a window bounds the keys from below, sequences of a pass may be of any
// length and sit anywhere in the row buffers, and the output leaves times the head's gate.
//
// TMEM (512 columns per block, one block per SM): score buffer b at columns 128 b (P_j overwrites its first 64
// as packed pairs), O of the same step at columns 256 + 128 b.
//
// Every mbarrier wait is bounded: on expiry the block records a code in the device error word, all roles leave
// their loops, nothing is stored, the TMEM columns are freed and the kernel returns.
#include <cuda.h>

#include <algorithm>

#include "device_utils.cuh"
#include "hybrid.h"
#include "tc_ptx.cuh"

namespace {

constexpr float NEG_BIG = -1.0e30f;
enum : uint32_t { ERR_LAT_Q = 0x61, ERR_LAT_K, ERR_LAT_V, ERR_LAT_S, ERR_LAT_P, ERR_LAT_O, ERR_LAT_FREE, ERR_LAT_KE, ERR_LAT_VE };
constexpr int TM_COLS = 512;
constexpr int BOX = 16384; // 128 rows x 64 bf16
constexpr int NTHREADS = 192;

struct Bars {
    uint64_t q_full;
    uint64_t k_full[2], k_empty[2], v_full[2], v_empty[2];
    uint64_t s_full[2], p_full[2], o_full[2], s_free[2];
};

// VB: 64-column boxes of a value row.
template <int VB>
__global__ void __launch_bounds__(NTHREADS, 1)
latent_prefill_tc_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_k,
                         const __grid_constant__ CUtensorMap tm_r, const __grid_constant__ CUtensorMap tm_v, LatentDims d, SeqMap sm,
                         float scale_log2e, const float *__restrict__ gate, __nv_bfloat16 *__restrict__ out, uint32_t *__restrict__ dev_err) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ __align__(8) Bars bars;
    __shared__ uint32_t tmem_slot;
    __shared__ int abort_flag;

    const int h = blockIdx.x, sidx = blockIdx.y, qt = blockIdx.z;
    const int tid = threadIdx.x, warp = tid >> 5;
    pdl_wait();
    const int n = sm.n[sidx];
    if (qt * 128 >= n) return; // the whole block
    const int nbn = (d.dim_p + 63) >> 6, kb = nbn + 1; // boxes of a key: unrotated ones, one rotated
    const uint32_t base = (tc::smem_u32(smem_raw) + 1023u) & ~1023u;
    const uint32_t sQ = base, sK = sQ + kb * BOX, sV = sK + 2 * kb * BOX;
    auto bar = [&](const uint64_t &x) { return tc::smem_u32(&x); };

    if (tid == 0) {
        abort_flag = 0;
        tc::mbar_init(bar(bars.q_full), 1);
        for (int i = 0; i < 2; ++i) {
            tc::mbar_init(bar(bars.k_full[i]), 1);
            tc::mbar_init(bar(bars.k_empty[i]), 1);
            tc::mbar_init(bar(bars.v_full[i]), 1);
            tc::mbar_init(bar(bars.v_empty[i]), 1);
            tc::mbar_init(bar(bars.s_full[i]), 1);
            tc::mbar_init(bar(bars.p_full[i]), 128); // every softmax thread
            tc::mbar_init(bar(bars.o_full[i]), 1);
            tc::mbar_init(bar(bars.s_free[i]), 128);
        }
        tc::fence_mbar_init();
    }
    if (warp == 1) tc::tmem_alloc(tc::smem_u32(&tmem_slot), TM_COLS);
    tc::tc_fence_before_sync();
    __syncthreads();
    tc::tc_fence_after_sync();
    pdl_trigger(); // only now: a dependent block must not take this one's tensor memory
    const uint32_t tmem_base = *reinterpret_cast<volatile uint32_t *>(&tmem_slot);

    // keys in gathered-row coordinates of the sequence: [kbeg, kend)
    const int past = sm.past[sidx], kpos0 = sm.kpos0[sidx], row0 = sm.row0[sidx], krow0 = sm.krow0[sidx];
    const int q_first = past + qt * 128, q_last = past + min(n, qt * 128 + 128) - 1;
    const int kbeg = (d.window ? max(0, q_first - d.window + 1) : 0) - kpos0, kend = q_last - kpos0 + 1;
    const int n_tiles = (kend - kbeg + 127) >> 7;

    if (warp == 0) {
        // ---- copies ----
        if (tc::elect_one()) {
            tc::mbar_expect_tx(bar(bars.q_full), kb * BOX);
            for (int i = 0; i < nbn; ++i) tc::tma_load_3d(sQ + i * BOX, &tm_q, i * 64, h, row0 + qt * 128, bar(bars.q_full));
            tc::tma_load_3d(sQ + nbn * BOX, &tm_q, d.dim_p, h, row0 + qt * 128, bar(bars.q_full));
        }
        __syncwarp();
        for (int j = 0; j < n_tiles; ++j) {
            const int st = j & 1, u = j >> 1, y = krow0 + kbeg + j * 128;
            if (j >= 2 && !tc::mbar_wait(bar(bars.k_empty[st]), (u - 1) & 1, &abort_flag, dev_err, ERR_LAT_KE)) break;
            if (tc::elect_one()) {
                const uint32_t dst = sK + st * kb * BOX;
                tc::mbar_expect_tx(bar(bars.k_full[st]), kb * BOX);
                for (int i = 0; i < nbn; ++i) tc::tma_load_3d(dst + i * BOX, &tm_k, i * 64, h, y, bar(bars.k_full[st]));
                tc::tma_load_2d(dst + nbn * BOX, &tm_r, 0, y, bar(bars.k_full[st]));
            }
            __syncwarp();
            if (j >= 2 && !tc::mbar_wait(bar(bars.v_empty[st]), (u - 1) & 1, &abort_flag, dev_err, ERR_LAT_VE)) break;
            if (tc::elect_one()) {
                tc::mbar_expect_tx(bar(bars.v_full[st]), VB * BOX);
#pragma unroll
                for (int i = 0; i < VB; ++i) tc::tma_load_3d(sV + (st * VB + i) * BOX, &tm_v, i * 64, h, y, bar(bars.v_full[st]));
            }
            __syncwarp();
        }
    } else if (warp == 1) {
        // ---- MMA issue: S_j as early as its buffer and K tile allow, then O_{j-1} once P_{j-1} is written ----
        constexpr uint32_t idesc_s = tc::umma_idesc_f16(128, 128) | tc::UMMA_BF16;
        constexpr uint32_t idesc_o = tc::umma_idesc_f16_bmn(128, 64) | tc::UMMA_BF16;
        const int steps_n = d.dim_p >> 4, steps_r = d.rot_p >> 4;
        const uint64_t dq = tc::umma_desc_sw128(sQ);
        bool ok = tc::mbar_wait(bar(bars.q_full), 0, &abort_flag, dev_err, ERR_LAT_Q);
        for (int j = 0; ok && j <= n_tiles; ++j) {
            if (j < n_tiles) {
                const int bf = j & 1, u = j >> 1;
                if (j >= 2) ok = tc::mbar_wait(bar(bars.s_free[bf]), (u - 1) & 1, &abort_flag, dev_err, ERR_LAT_FREE);
                if (ok) ok = tc::mbar_wait(bar(bars.k_full[bf]), u & 1, &abort_flag, dev_err, ERR_LAT_K);
                if (!ok) break;
                tc::tc_fence_after_sync();
                if (tc::elect_one()) {
                    const uint64_t dk = tc::umma_desc_sw128(sK + bf * kb * BOX);
                    for (int k = 0; k < steps_n; ++k) { // 16 columns a step, four steps a box
                        const uint64_t off = (uint64_t)((k >> 2) * (BOX >> 4) + (k & 3) * 2);
                        tc::umma_f16_ss(tmem_base + bf * 128, dq + off, dk + off, idesc_s, k != 0);
                    }
                    for (int k = 0; k < steps_r; ++k) {
                        const uint64_t off = (uint64_t)(nbn * (BOX >> 4) + k * 2);
                        tc::umma_f16_ss(tmem_base + bf * 128, dq + off, dk + off, idesc_s, 1u);
                    }
                    tc::umma_commit(bar(bars.s_full[bf]));
                    tc::umma_commit(bar(bars.k_empty[bf]));
                }
                __syncwarp();
            }
            if (j >= 1) {
                const int jp = j - 1, bp = jp & 1;
                ok = tc::mbar_wait(bar(bars.p_full[bp]), (jp >> 1) & 1, &abort_flag, dev_err, ERR_LAT_P);
                if (ok) ok = tc::mbar_wait(bar(bars.v_full[bp]), (jp >> 1) & 1, &abort_flag, dev_err, ERR_LAT_V);
                if (!ok) break;
                tc::tc_fence_after_sync();
                if (tc::elect_one()) {
#pragma unroll
                    for (int i = 0; i < VB; ++i) {
                        const uint64_t dv = tc::umma_desc_sw128_mn64(sV + (bp * VB + i) * BOX);
#pragma unroll
                        for (int k = 0; k < 8; ++k) // 16 keys per MMA: 8 TMEM columns of P, 2048 bytes of V
                            tc::umma_f16_ts(tmem_base + 256 + bp * 128 + i * 64, tmem_base + bp * 128 + 8 * k, dv + (uint64_t)(k * (2048 >> 4)),
                                            idesc_o, k != 0);
                    }
                    tc::umma_commit(bar(bars.o_full[bp]));
                    tc::umma_commit(bar(bars.v_empty[bp]));
                }
                __syncwarp();
            }
        }
    } else {
        // ---- softmax and the running output: thread = query row = TMEM lane ----
        const int quad = warp & 3, row = quad * 32 + (tid & 31);
        const uint32_t lane_base = tmem_base + ((uint32_t)(quad * 32) << 16);
        const int s_row = qt * 128 + row;
        const bool row_valid = s_row < n;
        const int a_pos = past + s_row;
        const int lo = (d.window ? max(0, a_pos - d.window + 1) : 0) - kpos0 - kbeg, hi = a_pos - kpos0 - kbeg; // visible keys, inclusive
        float m = NEG_BIG, l = 0.0f, corr_prev = 1.0f, acc[64 * VB];
#pragma unroll
        for (int e = 0; e < 64 * VB; ++e) acc[e] = 0.0f;
        bool ok = true;
        auto fold_output = [&](int bp, float c) { // acc = acc * c + O_tile
#pragma unroll
            for (int i = 0; i < VB; ++i) {
                uint32_t v[64];
                tc::tmem_ld_x64(lane_base + 256 + bp * 128 + i * 64, v);
#pragma unroll
                for (int e = 0; e < 64; ++e) acc[i * 64 + e] = fmaf(acc[i * 64 + e], c, __uint_as_float(v[e]));
            }
        };
        for (int j = 0; j < n_tiles; ++j) {
            const int bf = j & 1;
            const uint32_t sbuf = lane_base + bf * 128;
            ok = tc::mbar_wait(bar(bars.s_full[bf]), (j >> 1) & 1, &abort_flag, dev_err, ERR_LAT_S);
            if (!ok) break;
            tc::tc_fence_after_sync();
            // columns [c0, c1) of this tile the row may attend to; only the tiles at the two edges of the
            // window (and rows past the sequence) need the mask
            const int c0 = max(0, lo - j * 128), c1 = row_valid ? min(128, hi - j * 128 + 1) : 0;
            const bool full = __all_sync(0xffffffffu, c0 == 0 && c1 == 128);
            float mx[4] = {NEG_BIG, NEG_BIG, NEG_BIG, NEG_BIG};
#pragma unroll 1
            for (int hf = 0; hf < 2; ++hf) { // pass 1: row maximum
                uint32_t v[64];
                tc::tmem_ld_x64(sbuf + 64 * hf, v);
                if (full) {
#pragma unroll
                    for (int e = 0; e < 64; e += 8) {
                        mx[0] = tc::fmax3(mx[0], __uint_as_float(v[e]), __uint_as_float(v[e + 1]));
                        mx[1] = tc::fmax3(mx[1], __uint_as_float(v[e + 2]), __uint_as_float(v[e + 3]));
                        mx[2] = tc::fmax3(mx[2], __uint_as_float(v[e + 4]), __uint_as_float(v[e + 5]));
                        mx[3] = tc::fmax3(mx[3], __uint_as_float(v[e + 6]), __uint_as_float(v[e + 7]));
                    }
                } else {
#pragma unroll
                    for (int e = 0; e < 64; ++e)
                        if (64 * hf + e >= c0 && 64 * hf + e < c1) mx[e & 3] = fmaxf(mx[e & 3], __uint_as_float(v[e]));
                }
            }
            const float mloc = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3]));
            const float m_new = mloc > NEG_BIG ? fmaxf(m, mloc * scale_log2e) : m;
            const float corr = tc::ex2_approx(m - m_new);
            if (j >= 1) { // the previous step's P V has had pass 1 to finish
                ok = tc::mbar_wait(bar(bars.o_full[bf ^ 1]), ((j - 1) >> 1) & 1, &abort_flag, dev_err, ERR_LAT_O);
                if (!ok) break;
                tc::tc_fence_after_sync();
                fold_output(bf ^ 1, corr_prev);
                tc::tc_fence_before_sync();
                tc::mbar_arrive(bar(bars.s_free[bf ^ 1])); // that buffer may take S_{j+1}
            }
            float ls[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll 1
            for (int hf = 0; hf < 2; ++hf) { // pass 2: p = 2^(s*scale - max) as bf16 pairs over the scores
                uint32_t v[64], o[32];
                tc::tmem_ld_x64(sbuf + 64 * hf, v);
#pragma unroll
                for (int e = 0; e < 64; e += 2) {
                    float p0 = tc::ex2_approx(fmaf(__uint_as_float(v[e]), scale_log2e, -m_new));
                    float p1 = tc::ex2_approx(fmaf(__uint_as_float(v[e + 1]), scale_log2e, -m_new));
                    if (!full) {
                        if (64 * hf + e < c0 || 64 * hf + e >= c1) p0 = 0.0f;
                        if (64 * hf + e + 1 < c0 || 64 * hf + e + 1 >= c1) p1 = 0.0f;
                    }
                    ls[(e >> 1) & 3] += p0 + p1;
                    o[e >> 1] = pack_bf16x2(p0, p1);
                }
                tc::tmem_st_x32(sbuf + 32 * hf, o);
            }
            tc::tmem_st_wait();
            tc::tc_fence_before_sync();
            tc::mbar_arrive(bar(bars.p_full[bf]));
            l = l * corr + ((ls[0] + ls[1]) + (ls[2] + ls[3]));
            m = m_new;
            corr_prev = corr;
        }
        if (ok) {
            const int bl = (n_tiles - 1) & 1;
            ok = tc::mbar_wait(bar(bars.o_full[bl]), ((n_tiles - 1) >> 1) & 1, &abort_flag, dev_err, ERR_LAT_O);
            if (ok) {
                tc::tc_fence_after_sync();
                fold_output(bl, corr_prev);
            }
        }
        if (ok && row_valid) {
            const float f = gate[(size_t)(row0 + s_row) * d.heads + h] / l;
            uint4 *dst = reinterpret_cast<uint4 *>(out + ((size_t)(row0 + s_row) * d.heads + h) * d.vdim_p);
#pragma unroll
            for (int c = 0; c < 8 * VB; ++c) {
                if (8 * c >= d.vdim_p) break;
                dst[c] = make_uint4(pack_bf16x2(acc[8 * c] * f, acc[8 * c + 1] * f), pack_bf16x2(acc[8 * c + 2] * f, acc[8 * c + 3] * f),
                                    pack_bf16x2(acc[8 * c + 4] * f, acc[8 * c + 5] * f), pack_bf16x2(acc[8 * c + 6] * f, acc[8 * c + 7] * f));
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

// [rows][heads][cols] bf16 (rows row_w elements apart), one box = 128 rows x 64 columns of one head
int head_map(b200nn_ctx *ctx, const void *p, size_t cols, size_t heads, size_t rows, size_t row_w, CUtensorMap *out) {
    const cuuint64_t dim[3] = {cols, heads, rows};
    const cuuint64_t stride[2] = {cols * 2, row_w * 2};
    const cuuint32_t box[3] = {64, 1, 128}, ones[3] = {1, 1, 1};
    CUresult r = ((EncodeTiledFn)ctx->encode_tiled)(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, (void *)p, dim, stride, box, ones,
                                                    CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
                                                    CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) return set_error(ctx, B200NN_ERR_CUDA, "cuTensorMapEncodeTiled (latent attention) failed: " + std::to_string((int)r));
    return B200NN_OK;
}

template <int VB>
int launch_vb(b200nn_ctx *ctx, const LatentDims &d, const CUtensorMap &tq, const CUtensorMap &tk, const CUtensorMap &tr, const CUtensorMap &tv,
              const SeqMap &sm, const float *gate, __nv_bfloat16 *out) {
    auto kern = latent_prefill_tc_kernel<VB>;
    const int kb = (d.dim_p + 63) / 64 + 1;
    const int smem = (3 * kb + 2 * VB) * BOX + 1024;
    static bool attr_done[16] = {};
    if (!attr_done[ctx->device & 15]) {
        CK(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (9 + 2 * VB) * BOX + 1024));
        prefer_max_smem(kern);
        attr_done[ctx->device & 15] = true;
    }
    const dim3 grid(d.heads, sm.n_seq, (sm.max_n + 127) / 128);
    CK(ctx, launch_pdl(ctx, kern, grid, dim3(NTHREADS), (size_t)smem, tq, tk, tr, tv, d, sm, d.scale * 1.4426950408889634f, gate, out, ctx->dev_err));
    CK_LAUNCH(ctx, "latent_prefill_tc_kernel");
    return B200NN_OK;
}

}  // namespace

bool latent_prefill_tc_supported(const b200nn_ctx *ctx, const LatentDims &d) {
    return ctx->attn_tc && ctx->encode_tiled && d.dim_p <= 128 && d.rot_p <= 64 && d.vdim_p <= 128;
}

int launch_latent_prefill_tc(b200nn_ctx *ctx, const LatentDims &d, int n_rows, const __nv_bfloat16 *q, const __nv_bfloat16 *kvx,
                             const __nv_bfloat16 *lin, const SeqMap &sm, const float *gate, __nv_bfloat16 *out) {
    if (sm.n_seq > 65535 || (sm.max_n + 127) / 128 > 65535) return set_error(ctx, B200NN_ERR_SHAPE, "latent attention: more than 65535 sequences or query tiles");
    CUtensorMap tq, tk, tr, tv;
    TRY(head_map(ctx, q, d.head_w(), d.heads, n_rows, (size_t)d.heads * d.head_w(), &tq));
    TRY(head_map(ctx, kvx, d.dim_p, d.heads, sm.k_rows, d.kv_w(), &tk));
    TRY(head_map(ctx, kvx + (size_t)d.heads * d.dim_p, d.vdim_p, d.heads, sm.k_rows, d.kv_w(), &tv));
    {   // the shared rotated columns: [k_rows][rot_p], rows ld apart
        const cuuint64_t dim[2] = {(cuuint64_t)d.rot_p, (cuuint64_t)sm.k_rows};
        const cuuint64_t stride[1] = {(cuuint64_t)d.ld() * 2};
        const cuuint32_t box[2] = {64, 128}, ones[2] = {1, 1};
        CUresult r = ((EncodeTiledFn)ctx->encode_tiled)(&tr, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, (void *)(lin + d.rank_p), dim, stride, box, ones,
                                                        CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
                                                        CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
        if (r != CUDA_SUCCESS) return set_error(ctx, B200NN_ERR_CUDA, "cuTensorMapEncodeTiled (rotated keys) failed: " + std::to_string((int)r));
    }
    return d.vdim_p <= 64 ? launch_vb<1>(ctx, d, tq, tk, tr, tv, sm, gate, out) : launch_vb<2>(ctx, d, tq, tk, tr, tv, sm, gate, out);
}
