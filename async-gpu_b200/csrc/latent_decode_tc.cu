// Decode attention over cached latents on the tensor cores (tcgen05), bfloat16.
//
// All heads of a sequence read the same cache rows, so the product is turned around: the keys are the MMA's 128
// rows and the heads its columns,
//     S^T [128 keys x heads]  = rows [128 x (rank | rot)] . (query latents | rotated query)^T
//     O^T [rank x heads]     += rows^T [rank x 128] . P [128 x heads]
// with the cache tile in shared memory serving both: K-major A operand of the first product, MN-major A operand
// of the second.  A tile is read from memory once, whatever the number of heads in the block.
//
// Block = (key split, group of N heads, row), six warps:
//   warp 0      copies: the N queries once, then 128-row tiles of the ring through tensor maps, 128 latent columns
//               (two 64-column boxes, "a pair") at a time into a ring of pairs, the rotated columns beside them
//   warp 1      MMA issue: S^T pair by pair as they land, then O^T chunk by chunk; a pair is handed back as soon
//               as its chunk's products have retired, so the next tile's copies run under this tile's tail
//   warps 2..5  softmax: thread = key (TMEM lane), the heads in registers; maxima over keys by a transposing
//               butterfly and shared memory; P goes to shared memory as the K-major B operand.  The reference
//               maximum moves (and O^T is rescaled in place) only when a score exceeds it by more than 2^6.
// Tiles start at multiples of 128 positions, so a tile is contiguous in the ring; rows outside the window or
// past the position are masked.  With more than one split per row the blocks leave f32 partial sums and
// latent_merge_kernel adds them up.
//
// Every mbarrier wait is bounded (see attention_tc.cu).
#include <cuda.h>

#include <algorithm>

#include "device_utils.cuh"
#include "hybrid.h"
#include "tc_decode.cuh"

namespace {

constexpr float NEG_BIG = -1.0e30f;
enum : uint32_t { ERR_LD_Q = 0x71, ERR_LD_C, ERR_LD_R, ERR_LD_S, ERR_LD_P, ERR_LD_O, ERR_LD_CE, ERR_LD_RE };
constexpr int NTHREADS = 192;
constexpr int BOX = 16384, PAIR = 2 * BOX; // 128 rows x 64 bf16
constexpr int MAX_PAIRS = 6, MAX_TILE_PAIRS = 5; // ring; rank_p <= 640

struct Bars {
    uint64_t q_full, r_full, r_empty, s_full, p_full, o_full;
    uint64_t c_full[MAX_PAIRS], c_empty[MAX_PAIRS];
};

struct DecodeTcArgs {
    LatentDims d;
    RowMap rows;
    int ring, tile_pairs, ring_pairs, splits;
    float scale_log2e;
    __nv_bfloat16 *out;  // [row][head][rank_p], when splits == 1
    float *part_o, *part_ml; // [split][row][head][rank_p], [split][row][head][2]
    uint32_t *dev_err;
};

template <int N>
__global__ void __launch_bounds__(NTHREADS)
latent_decode_tc_kernel(const __grid_constant__ CUtensorMap tm_c, const __grid_constant__ CUtensorMap tm_r,
                        const __grid_constant__ CUtensorMap tm_ql, const __grid_constant__ CUtensorMap tm_qr, const DecodeTcArgs a) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ __align__(8) Bars bars;
    __shared__ __align__(16) float red[4][N];
    __shared__ uint32_t tmem_slot;
    __shared__ int abort_flag;
    constexpr int QBOX = N * 128; // N query rows x 64 columns

    const LatentDims &d = a.d;
    const int split = blockIdx.x, h0 = blockIdx.y * N, row = blockIdx.z, n_rows = gridDim.z;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int nc = (d.rank_p + 63) >> 6, tp = a.tile_pairs, np = a.ring_pairs;
    const uint32_t base = (tc::smem_u32(smem_raw) + 1023u) & ~1023u;
    uint8_t *gen_base = smem_raw + (base - tc::smem_u32(smem_raw));
    const uint32_t sC = base, sR = sC + np * PAIR, sQ = sR + BOX, sP = sQ + (nc + 1) * QBOX;
    auto bar = [&](const uint64_t &x) { return tc::smem_u32(&x); };
    // TMEM columns: S^T in 0 .. N-1, O^T chunk i from N (1 + i) on
    const uint32_t need = N * (1 + tp);
    const uint32_t cols = need <= 32 ? 32 : need <= 64 ? 64 : need <= 128 ? 128 : 256;

    if (tid == 0) {
        abort_flag = 0;
        tc::mbar_init(bar(bars.q_full), 1);
        tc::mbar_init(bar(bars.r_full), 1);
        tc::mbar_init(bar(bars.r_empty), 1);
        tc::mbar_init(bar(bars.s_full), 1);
        tc::mbar_init(bar(bars.p_full), 128);
        tc::mbar_init(bar(bars.o_full), 1);
        for (int i = 0; i < np; ++i) {
            tc::mbar_init(bar(bars.c_full[i]), 1);
            tc::mbar_init(bar(bars.c_empty[i]), 1);
        }
        tc::fence_mbar_init();
    }
    if (tid == 32) {
        tc::prefetch_tmap(&tm_c);
        tc::prefetch_tmap(&tm_r);
        tc::prefetch_tmap(&tm_ql);
        tc::prefetch_tmap(&tm_qr);
    }
    pdl_wait();
    if (warp == 1) tc::tmem_alloc(tc::smem_u32(&tmem_slot), cols);
    tc::tc_fence_before_sync();
    __syncthreads();
    tc::tc_fence_after_sync();
    pdl_trigger(); // only now: a dependent block must not take this one's tensor memory
    const uint32_t tmem_base = *reinterpret_cast<volatile uint32_t *>(&tmem_slot);

    const int pos = row_pos(a.rows, row), slot = row_slot(a.rows, row);
    const int first = d.window ? max(0, pos - d.window + 1) : 0;
    const int t_first = first >> 7, t_all = (pos >> 7) - t_first + 1;
    const int per = (t_all + a.splits - 1) / a.splits;
    const int t0 = t_first + split * per, n_tiles = max(0, min(per, t_all - split * per));

    if (warp == 0) {
        // ---- copies ----
        if (n_tiles > 0 && tc::elect_one()) {
            tc::mbar_expect_tx(bar(bars.q_full), (nc + 1) * QBOX);
            for (int i = 0; i < nc; ++i) tc::tma_load_2d(sQ + i * QBOX, &tm_ql, i * 64, row * d.heads + h0, bar(bars.q_full));
            tc::tma_load_2d(sQ + nc * QBOX, &tm_qr, d.dim_p, row * d.heads + h0, bar(bars.q_full));
        }
        __syncwarp();
        int s = 0;
        uint32_t ph = 1; // parity already complete on a fresh barrier
        bool ok = true;
        for (int j = 0; ok && j < n_tiles; ++j) {
            const int y = slot * a.ring + (int)(((long long)(t0 + j) * 128) % a.ring);
            for (int i = 0; i < tp; ++i) {
                ok = tc::mbar_wait(bar(bars.c_empty[s]), ph, &abort_flag, a.dev_err, ERR_LD_CE);
                if (!ok) break;
                if (tc::elect_one()) {
                    const bool two = 2 * i + 1 < nc;
                    tc::mbar_expect_tx(bar(bars.c_full[s]), two ? PAIR : BOX);
                    tc::tma_load_2d(sC + s * PAIR, &tm_c, i * 128, y, bar(bars.c_full[s]));
                    if (two) tc::tma_load_2d(sC + s * PAIR + BOX, &tm_c, i * 128 + 64, y, bar(bars.c_full[s]));
                }
                __syncwarp();
                if (++s == np) { s = 0; ph ^= 1; }
            }
            if (!ok) break;
            ok = tc::mbar_wait(bar(bars.r_empty), (j & 1) ^ 1, &abort_flag, a.dev_err, ERR_LD_RE);
            if (!ok) break;
            if (tc::elect_one()) {
                tc::mbar_expect_tx(bar(bars.r_full), BOX);
                tc::tma_load_2d(sR, &tm_r, 0, y, bar(bars.r_full));
            }
            __syncwarp();
        }
    } else if (warp == 1) {
        // ---- MMA issue ----
        constexpr uint32_t idesc_s = tc::umma_idesc_f16(128, N) | tc::UMMA_BF16;
        constexpr uint32_t idesc_o = tc::umma_idesc_f16(128, N) | tc::UMMA_BF16 | (1u << 15); // A MN-major
        const uint64_t dq = tc::umma_desc_sw128(sQ), dp = tc::umma_desc_sw128(sP);
        bool ok = n_tiles == 0 || tc::mbar_wait(bar(bars.q_full), 0, &abort_flag, a.dev_err, ERR_LD_Q);
        int s = 0;
        uint32_t ph = 0;
        for (int j = 0; ok && j < n_tiles; ++j) {
            const int s_tile = s;
            for (int i = 0; i < tp; ++i) {
                ok = tc::mbar_wait(bar(bars.c_full[s]), ph, &abort_flag, a.dev_err, ERR_LD_C);
                if (!ok) break;
                tc::tc_fence_after_sync();
                if (tc::elect_one()) {
                    const uint64_t dc = tc::umma_desc_sw128(sC + s * PAIR);
                    const int steps = min(8, (d.rank_p - i * 128) >> 4);
                    for (int k = 0; k < steps; ++k) // 16 columns a step, four steps a box
                        tc::umma_f16_ss(tmem_base, dc + (uint64_t)((k >> 2) * (BOX >> 4) + (k & 3) * 2),
                                        dq + (uint64_t)((2 * i + (k >> 2)) * (QBOX >> 4) + (k & 3) * 2), idesc_s, (i | k) != 0);
                }
                __syncwarp();
                if (++s == np) { s = 0; ph ^= 1; }
            }
            if (ok) ok = tc::mbar_wait(bar(bars.r_full), j & 1, &abort_flag, a.dev_err, ERR_LD_R);
            if (!ok) break;
            tc::tc_fence_after_sync();
            if (tc::elect_one()) {
                const uint64_t dr = tc::umma_desc_sw128(sR);
                for (int k = 0; k < (d.rot_p >> 4); ++k)
                    tc::umma_f16_ss(tmem_base, dr + 2 * k, dq + (uint64_t)(nc * (QBOX >> 4) + 2 * k), idesc_s, 1u);
                tc::umma_commit(bar(bars.s_full));
                tc::umma_commit(bar(bars.r_empty));
            }
            __syncwarp();
            ok = tc::mbar_wait(bar(bars.p_full), j & 1, &abort_flag, a.dev_err, ERR_LD_P);
            if (!ok) break;
            tc::tc_fence_after_sync();
            int sp = s_tile;
            for (int i = 0; i < tp; ++i) {
                if (tc::elect_one()) {
                    // rank chunk i: 128 M values in two 64-wide blocks BOX apart (leading byte offset)
                    const uint64_t dc = (tc::umma_desc_sw128(sC + sp * PAIR) & ~((uint64_t)0x3fff << 16)) | ((uint64_t)(BOX >> 4) << 16);
#pragma unroll
                    for (int k = 0; k < 8; ++k) // 16 keys a step: 2048 bytes of the tile, 32 bytes of P
                        tc::umma_f16_ss(tmem_base + N * (1 + i), dc + (uint64_t)(k * (2048 >> 4)),
                                        dp + (uint64_t)((k >> 2) * (QBOX >> 4) + (k & 3) * 2), idesc_o, (j | k) != 0);
                    tc::umma_commit(bar(bars.c_empty[sp]));
                }
                __syncwarp();
                if (++sp == np) sp = 0;
            }
            if (j == n_tiles - 1 && tc::elect_one()) tc::umma_commit(bar(bars.o_full));
            __syncwarp();
        }
    } else {
        // ---- softmax and output: thread = key of the tile, later latent column of a chunk ----
        const int quad = warp & 3, key = quad * 32 + lane;
        const uint32_t lane_base = tmem_base + ((uint32_t)(quad * 32) << 16);
        uint8_t *p_row = gen_base + (sP - base) + (key >> 6) * QBOX + (key & 7) * 2; // + swizzled 16-byte chunk of (head, key)
        const int chunk = (key & 63) >> 3;
        float m[N], l[N];
#pragma unroll
        for (int h = 0; h < N; ++h) m[h] = NEG_BIG, l[h] = 0.0f;
        bool ok = true;
        for (int j = 0; j < n_tiles; ++j) {
            ok = tc::mbar_wait(bar(bars.s_full), j & 1, &abort_flag, a.dev_err, ERR_LD_S);
            ok = !tc::bar_softmax_any(!ok); // all four warps go on or none does; red is free again
            if (!ok) break;
            tc::tc_fence_after_sync();
            float v[N], t[N];
            tc::tmem_ld_cols<N>(lane_base, v);
            const int kp = (t0 + j) * 128 + key;
            const bool vis = kp >= first && kp <= pos;
#pragma unroll
            for (int h = 0; h < N; ++h) t[h] = v[h] = vis ? v[h] * a.scale_log2e : -INFINITY;
            tc::reduce_columns<N, true>(t);
            if (N == 32) red[quad][lane] = t[0];
            else if (!(lane & 1)) red[quad][lane >> 1] = t[0];
            tc::bar_softmax();
            bool moved = false;
#pragma unroll
            for (int h = 0; h < N; ++h) {
                const float mx = fmaxf(fmaxf(red[0][h], red[1][h]), fmaxf(red[2][h], red[3][h]));
                const float mn = mx > m[h] + 6.0f ? mx : m[h]; // the same in every thread
                t[h] = tc::ex2_approx(m[h] - mn);
                moved |= mn != m[h];
                m[h] = mn;
            }
            if (moved) {
#pragma unroll
                for (int h = 0; h < N; ++h) l[h] *= t[h];
                if (j > 0) { // the products of the previous tiles have retired (S^T of this one was issued after them)
                    for (int i = 0; i < tp; ++i)
#pragma unroll
                        for (int c = 0; c < N; c += 16) {
                            uint32_t o[16];
                            tc::tmem_ld_x16(lane_base + N * (1 + i) + c, o);
#pragma unroll
                            for (int e = 0; e < 16; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * t[c + e]);
                            tc::tmem_st_x16(lane_base + N * (1 + i) + c, o);
                        }
                    tc::tmem_st_wait();
                }
            }
#pragma unroll
            for (int h = 0; h < N; ++h) {
                const float p = tc::ex2_approx(v[h] - m[h]);
                l[h] += p;
                *reinterpret_cast<__nv_bfloat16 *>(p_row + h * 128 + ((chunk ^ (h & 7)) << 4)) = __float2bfloat16_rn(p);
            }
            tc::fence_proxy_async_smem();
            tc::tc_fence_before_sync();
            tc::mbar_arrive(bar(bars.p_full));
        }
        tc::bar_softmax();
        if (ok) { // sums over the keys
            tc::reduce_columns<N, false>(l);
            if (N == 32) red[quad][lane] = l[0];
            else if (!(lane & 1)) red[quad][lane >> 1] = l[0];
        }
        tc::bar_softmax();
        if (ok && n_tiles > 0) {
            ok = tc::mbar_wait(bar(bars.o_full), 0, &abort_flag, a.dev_err, ERR_LD_O);
            tc::tc_fence_after_sync();
        }
        if (ok) {
#pragma unroll
            for (int h = 0; h < N; ++h) l[h] = (red[0][h] + red[1][h]) + (red[2][h] + red[3][h]);
            const size_t unit = (size_t)row * d.heads + h0;
            if (a.splits > 1 && tid < 64 + N && h0 + (tid - 64) < d.heads) { // one thread per head
                float mm = NEG_BIG, ll = 0.0f;
#pragma unroll
                for (int h = 0; h < N; ++h)
                    if (h == tid - 64) mm = m[h], ll = l[h];
                *reinterpret_cast<float2 *>(a.part_ml + ((size_t)split * n_rows * d.heads + unit + (tid - 64)) * 2) = make_float2(mm, n_tiles ? ll : 0.0f);
            }
            if (n_tiles > 0)
                for (int i = 0; i < tp; ++i) {
                    tc::tmem_ld_cols<N>(lane_base + N * (1 + i), m); // the maxima are not needed any more
                    const int c = i * 128 + key;
                    if (c < d.rank_p)
#pragma unroll
                        for (int h = 0; h < N; ++h)
                            if (h0 + h < d.heads) {
                                if (a.splits > 1) a.part_o[(((size_t)split * n_rows * d.heads) + unit + h) * d.rank_p + c] = m[h];
                                else a.out[(unit + h) * d.rank_p + c] = __float2bfloat16_rn(m[h] / l[h]);
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
    if (warp == 1) tc::tmem_dealloc(tmem_base, cols);
}

// Adds up the splits of one (head, row).
__global__ void __launch_bounds__(128)
latent_merge_kernel(const float *__restrict__ part_o, const float *__restrict__ part_ml, int splits, int heads, int rank_p,
                    __nv_bfloat16 *__restrict__ out) {
    pdl_trigger();
    pdl_wait();
    const size_t unit = (size_t)blockIdx.y * heads + blockIdx.x, stride = (size_t)gridDim.y * heads;
    float m = NEG_BIG;
    for (int s = 0; s < splits; ++s) m = fmaxf(m, __ldcg(part_ml + (s * stride + unit) * 2));
    float total = 0.0f;
    for (int s = 0; s < splits; ++s) {
        const float2 ml = __ldcg(reinterpret_cast<const float2 *>(part_ml) + s * stride + unit);
        total += ml.y * tc::ex2_approx(ml.x - m);
    }
    const float inv = 1.0f / total;
    for (int c = threadIdx.x * 4; c < rank_p; c += 512) {
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int s = 0; s < splits; ++s) {
            const float2 ml = __ldcg(reinterpret_cast<const float2 *>(part_ml) + s * stride + unit);
            if (ml.y == 0.0f) continue; // a split without keys left nothing
            const float f = tc::ex2_approx(ml.x - m) * inv;
            const float4 o = __ldcg(reinterpret_cast<const float4 *>(part_o + (s * stride + unit) * rank_p + c));
            acc.x = fmaf(f, o.x, acc.x); acc.y = fmaf(f, o.y, acc.y); acc.z = fmaf(f, o.z, acc.z); acc.w = fmaf(f, o.w, acc.w);
        }
        *reinterpret_cast<uint2 *>(out + unit * rank_p + c) = make_uint2(pack_bf16x2(acc.x, acc.y), pack_bf16x2(acc.z, acc.w));
    }
}

typedef CUresult (*EncodeTiledFn)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *, const cuuint64_t *,
                                  const cuuint64_t *, const cuuint32_t *, const cuuint32_t *, CUtensorMapInterleave,
                                  CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

// [rows][cols] bf16, rows ld elements apart, one box = box_rows x 64 columns
int matrix_map(b200nn_ctx *ctx, const void *p, size_t cols, size_t rows, size_t ld, int box_rows, CUtensorMap *out) {
    const cuuint64_t dim[2] = {cols, rows}, stride[1] = {ld * 2};
    const cuuint32_t box[2] = {64, (cuuint32_t)box_rows}, ones[2] = {1, 1};
    CUresult r = ((EncodeTiledFn)ctx->encode_tiled)(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, (void *)p, dim, stride, box, ones,
                                                    CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
                                                    CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) return set_error(ctx, B200NN_ERR_CUDA, "cuTensorMapEncodeTiled (latent decode) failed: " + std::to_string((int)r));
    return B200NN_OK;
}

int heads_per_block(const LatentDims &d) { return d.heads <= 16 ? 16 : 32; }
int tile_pairs_of(const LatentDims &d) { return (d.rank_p + 127) / 128; }
size_t fixed_smem(const LatentDims &d, int n) { return 1024 + BOX + (size_t)((d.rank_p + 63) / 64 + 1) * n * 128 + (size_t)n * 256; }
int ring_pairs_of(const LatentDims &d) {
    const int tp = tile_pairs_of(d);
    const size_t fixed = fixed_smem(d, heads_per_block(d));
    const int fit = (int)((227 * 1024 - 2048 - fixed) / PAIR);
    // two blocks per SM where a tile fits in half of it (they cover each other's softmax), else one with the deepest ring
    const int half = fixed + tp * PAIR <= 111 * 1024 ? (int)((111 * 1024 - fixed) / PAIR) : fit;
    return std::min({fit, half, 2 * tp, MAX_PAIRS});
}

// Key splits per row: the number that minimises (waves of blocks) x (tiles per block + about one tile's worth of
// start-up and partial sums).
int pick_splits(const b200nn_ctx *ctx, const LatentDims &d, int n_rows, int cap) {
    const int n = heads_per_block(d), hb = (d.heads + n - 1) / n;
    const int tiles = ((d.window ? std::min(d.window + 127, cap) : cap) + 127) / 128;
    const size_t smem = fixed_smem(d, n) + (size_t)ring_pairs_of(d) * PAIR;
    const long long per_wave = (long long)ctx->sm_count * std::max<size_t>(1, (227 * 1024) / (smem + 2048));
    int best = 1;
    double best_cost = 1e300;
    for (int s = 1; s <= std::min(tiles, 64); ++s) {
        const int per = (tiles + s - 1) / s;
        if (s > 1 && (tiles + s - 2) / (s - 1) == per) continue; // no shorter than with fewer splits
        const double waves = (double)(((long long)n_rows * hb * s + per_wave - 1) / per_wave);
        const double cost = waves * (per + (s > 1 ? 1.5 : 1.0));
        if (cost < best_cost) best_cost = cost, best = s;
    }
    return best;
}

template <int N>
int launch_n(b200nn_ctx *ctx, const DecodeTcArgs &a, const CUtensorMap &tc_, const CUtensorMap &tr, const CUtensorMap &tql, const CUtensorMap &tqr,
             int n_rows, size_t smem) {
    auto kern = latent_decode_tc_kernel<N>;
    static bool attr_done[16] = {};
    if (!attr_done[ctx->device & 15]) {
        CK(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024 - 2048));
        prefer_max_smem(kern);
        attr_done[ctx->device & 15] = true;
    }
    CK(ctx, launch_pdl(ctx, kern, dim3(a.splits, (a.d.heads + N - 1) / N, n_rows), dim3(NTHREADS), smem, tc_, tr, tql, tqr, a));
    CK_LAUNCH(ctx, "latent_decode_tc_kernel");
    return B200NN_OK;
}

}  // namespace

bool latent_decode_tc_supported(const b200nn_ctx *ctx, const LatentDims &d) {
    return ctx->attn_tc && ctx->encode_tiled && tile_pairs_of(d) <= MAX_TILE_PAIRS && d.rot_p <= 64 && ring_pairs_of(d) >= tile_pairs_of(d);
}

size_t latent_decode_tc_part_floats(const b200nn_ctx *ctx, const LatentDims &d, int n_rows, int cap) {
    const size_t s = pick_splits(ctx, d, n_rows, cap);
    return s > 1 ? s * n_rows * d.heads * (d.rank_p + 2) : 0;
}

// cache_rows: rows of the whole cache (slots x ring)
int launch_latent_decode_tc(b200nn_ctx *ctx, const LatentDims &d, const __nv_bfloat16 *q, const __nv_bfloat16 *qlat, const __nv_bfloat16 *cache,
                            int ring, size_t cache_rows, const RowMap &rows, int n_rows, int cap, __nv_bfloat16 *out, float *part) {
    const int n = heads_per_block(d);
    if (n_rows > 65535) return set_error(ctx, B200NN_ERR_SHAPE, "latent attention: more than 65535 rows");
    DecodeTcArgs a;
    a.d = d;
    a.rows = rows;
    a.ring = ring;
    a.tile_pairs = tile_pairs_of(d);
    a.ring_pairs = ring_pairs_of(d);
    a.splits = pick_splits(ctx, d, n_rows, cap);
    a.scale_log2e = d.scale * 1.4426950408889634f;
    a.out = out;
    a.part_o = part;
    a.part_ml = part ? part + (size_t)a.splits * n_rows * d.heads * d.rank_p : nullptr;
    a.dev_err = ctx->dev_err;
    CUtensorMap tcm, tr, tql, tqr;
    TRY(matrix_map(ctx, cache, d.rank_p, cache_rows, d.ld(), 128, &tcm));
    TRY(matrix_map(ctx, cache + d.rank_p, d.rot_p, cache_rows, d.ld(), 128, &tr));
    TRY(matrix_map(ctx, qlat, d.rank_p, (size_t)n_rows * d.heads, d.rank_p, n, &tql));
    TRY(matrix_map(ctx, q, d.head_w(), (size_t)n_rows * d.heads, d.head_w(), n, &tqr));
    const size_t smem = fixed_smem(d, n) + (size_t)a.ring_pairs * PAIR;
    TRY(n == 16 ? launch_n<16>(ctx, a, tcm, tr, tql, tqr, n_rows, smem) : launch_n<32>(ctx, a, tcm, tr, tql, tqr, n_rows, smem));
    if (a.splits > 1) {
        PREFER_SMEM_ONCE(latent_merge_kernel);
        CK(ctx, launch_pdl(ctx, latent_merge_kernel, dim3(d.heads, n_rows), dim3(128), 0, a.part_o, a.part_ml, a.splits, d.heads, d.rank_p, out));
        CK_LAUNCH(ctx, "latent_merge_kernel");
    }
    return B200NN_OK;
}
