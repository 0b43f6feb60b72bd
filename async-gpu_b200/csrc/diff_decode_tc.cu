// Decode step of differential attention on the tensor cores (tcgen05), bfloat16.
//
// The query heads of one key / value head read the same cache rows, and both maps the same values, so as in
// latent_decode_tc.cu the keys are the MMA's 128 rows and its N columns are (map, query head):
//     S^T [128 keys x N]  = keys [128 x (map 0 | map 1)] . Q^T      Q's row (map, head) is zero in the other map's columns
//     O^T [vdim x N]     += values^T [vdim x 128] . P [128 x N]
// A 128-position tile of a head's cache (keys of both maps, then values) is one contiguous block of memory, read once.
//
// Block = (key split, group of N / 2 query heads of a key / value head, row), six warps:
//   warp 0      copies: 128-row tiles of the cache into a ring of stages
//   warp 1      MMA issue: S^T of the next tile before O^T of this one, so that the softmax warps do not wait
//   warps 2..5  Q into shared memory; softmax: thread = key (TMEM lane), the columns in registers, maxima over keys by a
//               transposing butterfly and shared memory; P to shared memory as the K-major B operand (two buffers).  The
//               reference maximum moves (and O^T is rescaled in place) only when exceeded by more than 2^6.
// Tiles start at multiples of 128 positions; rows past the position are masked.  Every block leaves f32 partial sums;
// diff_merge_kernel adds the splits up, subtracts the maps and applies norm and gate.
//
// Every mbarrier wait is bounded (see attention_tc.cu).
#include <cuda.h>

#include <algorithm>

#include "device_utils.cuh"
#include "hybrid.h"
#include "tc_decode.cuh"

namespace {

constexpr float NEG_BIG = -1.0e30f, LOG2E = 1.4426950408889634f;
enum : uint32_t { ERR_DD_Q = 0x91, ERR_DD_K, ERR_DD_V, ERR_DD_S, ERR_DD_P, ERR_DD_O, ERR_DD_KE, ERR_DD_VE };
constexpr int NTHREADS = 192;
constexpr int BOX = 16384; // 128 rows x 64 bf16
constexpr int MAX_STAGES = 4;

struct Bars {
    uint64_t q_full, k_full[MAX_STAGES], k_empty[MAX_STAGES], v_full[MAX_STAGES], v_empty[MAX_STAGES];
    uint64_t s_full[2], p_full[2], o_full[2];
};

struct DiffDecodeArgs {
    DiffDims d;
    RowMap rows;
    const __nv_bfloat16 *q;
    int ldq, cap, splits, stages, kb, vb; // kb, vb: 64-column boxes of the keys (both maps) and of the values (even)
    float *part_o, *part_ml;              // [split][row][head][map][vdim_p], [split][row][head][map][2]
    uint32_t *dev_err;
};

template <int N>
__global__ void __launch_bounds__(NTHREADS)
diff_decode_tc_kernel(const __grid_constant__ CUtensorMap tm_c, const DiffDecodeArgs a) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ __align__(8) Bars bars;
    __shared__ __align__(16) float red[4][N];
    __shared__ uint32_t tmem_slot;
    __shared__ int abort_flag;
    constexpr int NH = N / 2;       // heads per block
    constexpr int QBOX = N * 128;   // N rows x 64 columns
    constexpr int PBUF = 2 * QBOX;  // N rows x 128 keys

    const DiffDims &d = a.d;
    const int blocks_per_kv = (d.group() + NH - 1) / NH;
    const int split = blockIdx.x, kvh = blockIdx.y / blocks_per_kv, hg0 = (blockIdx.y % blocks_per_kv) * NH, row = blockIdx.z, n_rows = gridDim.z;
    const int h0 = kvh * d.group() + hg0, nh = min(NH, d.group() - hg0); // this block's query heads
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int ns = a.stages, tv = a.vb >> 1, stage_bytes = (a.kb + a.vb) * BOX;
    const uint32_t base = (tc::smem_u32(smem_raw) + 1023u) & ~1023u;
    uint8_t *gen_base = smem_raw + (base - tc::smem_u32(smem_raw));
    const uint32_t sQ = base + ns * stage_bytes, sP = sQ + a.kb * QBOX;
    auto bar = [&](const uint64_t &x) { return tc::smem_u32(&x); };
    // TMEM columns: S^T buffers at 0 and N, O^T chunk i from N (2 + i) on
    const uint32_t need = N * (2 + tv);
    const uint32_t cols = need <= 64 ? 64 : need <= 128 ? 128 : 256;

    if (tid == 0) {
        abort_flag = 0;
        tc::mbar_init(bar(bars.q_full), 128);
        for (int i = 0; i < ns; ++i) {
            tc::mbar_init(bar(bars.k_full[i]), 1);
            tc::mbar_init(bar(bars.k_empty[i]), 1);
            tc::mbar_init(bar(bars.v_full[i]), 1);
            tc::mbar_init(bar(bars.v_empty[i]), 1);
        }
        for (int i = 0; i < 2; ++i) {
            tc::mbar_init(bar(bars.s_full[i]), 1);
            tc::mbar_init(bar(bars.p_full[i]), 128);
            tc::mbar_init(bar(bars.o_full[i]), 1);
        }
        tc::fence_mbar_init();
    }
    if (tid == 32) tc::prefetch_tmap(&tm_c);
    pdl_wait();
    if (warp == 1) tc::tmem_alloc(tc::smem_u32(&tmem_slot), cols);
    tc::tc_fence_before_sync();
    __syncthreads();
    tc::tc_fence_after_sync();
    pdl_trigger(); // only now: a dependent block must not take this one's tensor memory
    const uint32_t tmem_base = *reinterpret_cast<volatile uint32_t *>(&tmem_slot);

    const int pos = row_pos(a.rows, row);
    const int crow = (row_slot(a.rows, row) * d.kv_heads + kvh) * a.cap; // cache row of position 0
    const int t_all = (pos >> 7) + 1, per = (t_all + a.splits - 1) / a.splits;
    const int t0 = split * per, n_tiles = max(0, min(per, t_all - t0));

    if (warp == 0) {
        // ---- copies ----
        int s = 0;
        uint32_t ph = 1; // parity already complete on a fresh barrier
        for (int j = 0; j < n_tiles; ++j) {
            const int y = crow + (t0 + j) * 128;
            if (!tc::mbar_wait(bar(bars.k_empty[s]), ph, &abort_flag, a.dev_err, ERR_DD_KE)) break;
            if (tc::elect_one()) {
                tc::mbar_expect_tx(bar(bars.k_full[s]), a.kb * BOX);
                for (int i = 0; i < a.kb; ++i) tc::tma_load_2d(base + s * stage_bytes + i * BOX, &tm_c, i * 64, y, bar(bars.k_full[s]));
            }
            __syncwarp();
            if (!tc::mbar_wait(bar(bars.v_empty[s]), ph, &abort_flag, a.dev_err, ERR_DD_VE)) break;
            if (tc::elect_one()) {
                tc::mbar_expect_tx(bar(bars.v_full[s]), a.vb * BOX);
                for (int i = 0; i < a.vb; ++i) // boxes past the row's end are filled with zeros
                    tc::tma_load_2d(base + s * stage_bytes + (a.kb + i) * BOX, &tm_c, 2 * d.dim_p + i * 64, y, bar(bars.v_full[s]));
            }
            __syncwarp();
            if (++s == ns) { s = 0; ph ^= 1; }
        }
    } else if (warp == 1) {
        // ---- MMA issue ----
        constexpr uint32_t idesc_s = tc::umma_idesc_f16(128, N) | tc::UMMA_BF16;
        constexpr uint32_t idesc_o = tc::umma_idesc_f16(128, N) | tc::UMMA_BF16 | (1u << 15); // A MN-major
        const uint64_t dq = tc::umma_desc_sw128(sQ);
        const int steps = (2 * d.dim_p) >> 4;
        int ks = 0, vs = 0;
        uint32_t kph = 0, vph = 0;
        auto issue_s = [&](int j) {
            bool ok = tc::mbar_wait(bar(bars.k_full[ks]), kph, &abort_flag, a.dev_err, ERR_DD_K);
            if (!ok) return false;
            tc::tc_fence_after_sync();
            if (tc::elect_one()) {
                const uint64_t dk = tc::umma_desc_sw128(base + ks * stage_bytes);
                for (int k = 0; k < steps; ++k) // 16 columns a step, four steps a box
                    tc::umma_f16_ss(tmem_base + (j & 1) * N, dk + (uint64_t)((k >> 2) * (BOX >> 4) + (k & 3) * 2),
                                    dq + (uint64_t)((k >> 2) * (QBOX >> 4) + (k & 3) * 2), idesc_s, k != 0);
                tc::umma_commit(bar(bars.s_full[j & 1]));
                tc::umma_commit(bar(bars.k_empty[ks]));
            }
            __syncwarp();
            if (++ks == ns) { ks = 0; kph ^= 1; }
            return true;
        };
        bool ok = n_tiles == 0 || (tc::mbar_wait(bar(bars.q_full), 0, &abort_flag, a.dev_err, ERR_DD_Q) && issue_s(0));
        for (int j = 0; ok && j < n_tiles; ++j) {
            if (j + 1 < n_tiles) ok = issue_s(j + 1); // its buffer was read before P of tile j - 1 arrived
            if (ok) ok = tc::mbar_wait(bar(bars.p_full[j & 1]), (j >> 1) & 1, &abort_flag, a.dev_err, ERR_DD_P);
            if (ok) ok = tc::mbar_wait(bar(bars.v_full[vs]), vph, &abort_flag, a.dev_err, ERR_DD_V);
            if (!ok) break;
            tc::tc_fence_after_sync();
            if (tc::elect_one()) {
                const uint64_t dp = tc::umma_desc_sw128(sP + (j & 1) * PBUF);
                for (int i = 0; i < tv; ++i) {
                    // value chunk i: 128 M values in two 64-wide blocks BOX apart (leading byte offset)
                    const uint64_t dv = (tc::umma_desc_sw128(base + vs * stage_bytes + (a.kb + 2 * i) * BOX) & ~((uint64_t)0x3fff << 16)) |
                                        ((uint64_t)(BOX >> 4) << 16);
#pragma unroll
                    for (int k = 0; k < 8; ++k) // 16 keys a step: 2048 bytes of the tile, 32 bytes of P
                        tc::umma_f16_ss(tmem_base + N * (2 + i), dv + (uint64_t)(k * (2048 >> 4)),
                                        dp + (uint64_t)((k >> 2) * (QBOX >> 4) + (k & 3) * 2), idesc_o, (j | k) != 0);
                }
                tc::umma_commit(bar(bars.v_empty[vs]));
                tc::umma_commit(bar(bars.o_full[j & 1]));
            }
            __syncwarp();
            if (++vs == ns) { vs = 0; vph ^= 1; }
        }
    } else {
        // ---- queries, softmax and output: thread = key of the tile, later value column of a chunk ----
        const int quad = warp & 3, key = quad * 32 + lane;
        const uint32_t lane_base = tmem_base + ((uint32_t)(quad * 32) << 16);
        if (n_tiles > 0) {
            // Q rows (map, head): 16-byte chunks of 8 columns, swizzled like a copied box
            for (int i = tid - 64; i < a.kb * N * 8; i += 128) {
                const int box = i / (N * 8), c = (i >> 3) % N, ch = i & 7, col = box * 64 + ch * 8, map = c / NH, hh = c % NH;
                uint4 v = make_uint4(0, 0, 0, 0);
                if (hh < nh && col >= map * d.dim_p && col < (map + 1) * d.dim_p)
                    v = *reinterpret_cast<const uint4 *>(a.q + (size_t)row * a.ldq + (size_t)(h0 + hh) * 2 * d.dim_p + col);
                *reinterpret_cast<uint4 *>(gen_base + (sQ - base) + box * QBOX + c * 128 + ((ch ^ (c & 7)) << 4)) = v;
            }
            tc::fence_proxy_async_smem();
            tc::mbar_arrive(bar(bars.q_full));
        }
        uint8_t *p_row = gen_base + (sP - base) + (key >> 6) * QBOX + (key & 7) * 2; // + buffer, + swizzled 16-byte chunk of (column, key)
        const int chunk = (key & 63) >> 3;
        // scores in units of log2: s * f, with a cap cap log2(e) tanh(s * f)
        const bool capped = d.cap > 0.0f;
        const float f = capped ? d.score_scale(pos) / d.cap * (2.0f * LOG2E) : d.score_scale(pos) * LOG2E, fc = d.cap * LOG2E;
        float m[N], l[N];
#pragma unroll
        for (int c = 0; c < N; ++c) m[c] = NEG_BIG, l[c] = 0.0f;
        bool ok = true;
        for (int j = 0; j < n_tiles; ++j) {
            ok = tc::mbar_wait(bar(bars.s_full[j & 1]), (j >> 1) & 1, &abort_flag, a.dev_err, ERR_DD_S);
            // P's buffer: the products of tile j - 2 have read it
            if (ok && j >= 2) ok = tc::mbar_wait(bar(bars.o_full[j & 1]), ((j >> 1) - 1) & 1, &abort_flag, a.dev_err, ERR_DD_O);
            ok = !tc::bar_softmax_any(!ok); // all four warps go on or none does; red is free again
            if (!ok) break;
            tc::tc_fence_after_sync();
            float v[N], t[N];
            tc::tmem_ld_cols<N>(lane_base + (j & 1) * N, v);
            const bool vis = (t0 + j) * 128 + key <= pos;
#pragma unroll
            for (int c = 0; c < N; ++c) {
                float s = v[c] * f;
                if (capped) { // 1 - 2 / (1 + e^2x)
                    float r;
                    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.0f + tc::ex2_approx(s)));
                    s = fc * fmaf(-2.0f, r, 1.0f);
                }
                t[c] = v[c] = vis ? s : -INFINITY;
            }
            tc::reduce_columns<N, true>(t);
            if (N == 32) red[quad][lane] = t[0];
            else if (!(lane & 1)) red[quad][lane >> 1] = t[0];
            tc::bar_softmax();
            bool moved = false;
#pragma unroll
            for (int c = 0; c < N; ++c) {
                const float mx = fmaxf(fmaxf(red[0][c], red[1][c]), fmaxf(red[2][c], red[3][c]));
                const float mn = mx > m[c] + 6.0f ? mx : m[c]; // the same in every thread
                t[c] = tc::ex2_approx(m[c] - mn);
                moved |= mn != m[c];
                m[c] = mn;
            }
            if (moved) {
#pragma unroll
                for (int c = 0; c < N; ++c) l[c] *= t[c];
                if (j > 0) {
                    ok = tc::mbar_wait(bar(bars.o_full[(j - 1) & 1]), ((j - 1) >> 1) & 1, &abort_flag, a.dev_err, ERR_DD_O);
                    if (ok) {
                        tc::tc_fence_after_sync();
                        for (int i = 0; i < tv; ++i)
#pragma unroll
                            for (int c = 0; c < N; c += 16) {
                                uint32_t o[16];
                                tc::tmem_ld_x16(lane_base + N * (2 + i) + c, o);
#pragma unroll
                                for (int e = 0; e < 16; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * t[c + e]);
                                tc::tmem_st_x16(lane_base + N * (2 + i) + c, o);
                            }
                        tc::tmem_st_wait();
                    }
                }
            }
#pragma unroll
            for (int c = 0; c < N; ++c) {
                const float p = tc::ex2_approx(v[c] - m[c]);
                l[c] += p;
                *reinterpret_cast<__nv_bfloat16 *>(p_row + (j & 1) * PBUF + c * 128 + ((chunk ^ (c & 7)) << 4)) = __float2bfloat16_rn(p);
            }
            tc::fence_proxy_async_smem();
            tc::tc_fence_before_sync();
            tc::mbar_arrive(bar(bars.p_full[j & 1]));
        }
        tc::bar_softmax();
        if (ok) { // sums over the keys
            tc::reduce_columns<N, false>(l);
            if (N == 32) red[quad][lane] = l[0];
            else if (!(lane & 1)) red[quad][lane >> 1] = l[0];
        }
        tc::bar_softmax();
        if (ok && n_tiles > 0) {
            ok = tc::mbar_wait(bar(bars.o_full[(n_tiles - 1) & 1]), ((n_tiles - 1) >> 1) & 1, &abort_flag, a.dev_err, ERR_DD_O);
            tc::tc_fence_after_sync();
        }
        if (ok) {
            const size_t unit0 = (((size_t)split * n_rows + row) * d.heads + h0) * 2;
            const int c0 = tid - 64; // one thread per column writes its maximum and sum
            if (c0 < N && c0 % NH < nh) {
                float mm = NEG_BIG;
#pragma unroll
                for (int c = 0; c < N; ++c)
                    if (c == c0) mm = m[c];
                const float ll = n_tiles ? (red[0][c0] + red[1][c0]) + (red[2][c0] + red[3][c0]) : 0.0f;
                *reinterpret_cast<float2 *>(a.part_ml + (unit0 + (c0 % NH) * 2 + c0 / NH) * 2) = make_float2(mm, ll);
            }
            if (n_tiles > 0)
                for (int i = 0; i < tv; ++i) {
                    tc::tmem_ld_cols<N>(lane_base + N * (2 + i), l); // the sums are not needed any more
                    const int e = i * 128 + key;
                    if (e < d.vdim_p)
#pragma unroll
                        for (int c = 0; c < N; ++c)
                            if (c % NH < nh) a.part_o[(unit0 + (c % NH) * 2 + c / NH) * d.vdim_p + e] = l[c];
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

// Adds up the splits of one (head, row), then the two maps, norm and gate.
__global__ void __launch_bounds__(128)
diff_merge_kernel(DiffDims d, const float *__restrict__ part_o, const float *__restrict__ part_ml, int splits, const float *__restrict__ gate, int gate_ld,
                  __nv_bfloat16 *__restrict__ out) {
    __shared__ float red[4];
    pdl_trigger();
    pdl_wait();
    const int h = blockIdx.x, row = blockIdx.y, tid = threadIdx.x;
    const size_t unit = ((size_t)row * d.heads + h) * 2, stride = (size_t)gridDim.y * d.heads * 2;
    float m[2] = {NEG_BIG, NEG_BIG}, total[2] = {0.0f, 0.0f};
    for (int s = 0; s < splits; ++s) {
        const float4 ml = __ldcg(reinterpret_cast<const float4 *>(part_ml + (s * stride + unit) * 2)); // (max, sum) of both maps
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const float mm = x ? ml.z : ml.x, ll = x ? ml.w : ml.y, mn = fmaxf(m[x], mm);
            total[x] = total[x] * tc::ex2_approx(m[x] - mn) + ll * tc::ex2_approx(mm - mn);
            m[x] = mn;
        }
    }
    const float inv[2] = {1.0f / total[0], -d.lambda / total[1]};
    float acc[4] = {0.f, 0.f, 0.f, 0.f}, ss = 0.0f; // vdim_p <= 512
    for (int s = 0; s < splits; ++s) {
        const float4 ml = __ldcg(reinterpret_cast<const float4 *>(part_ml + (s * stride + unit) * 2));
        if (ml.y == 0.0f) continue; // a split without keys left nothing
        const float f0 = tc::ex2_approx(ml.x - m[0]) * inv[0], f1 = tc::ex2_approx(ml.z - m[1]) * inv[1];
        const float *o = part_o + (s * stride + unit) * d.vdim_p;
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const int e = tid + 128 * c;
            if (e < d.vdim_p) acc[c] += f0 * __ldcg(o + e) + f1 * __ldcg(o + d.vdim_p + e);
        }
    }
#pragma unroll
    for (int c = 0; c < 4; ++c) ss = fmaf(acc[c], acc[c], ss); // columns past vdim are zero
    ss = warp_sum(ss);
    if ((tid & 31) == 0) red[tid >> 5] = ss;
    __syncthreads();
    ss = (red[0] + red[1]) + (red[2] + red[3]);
    const float f = (1.0f - d.diff) * sigmoid_f(gate[(size_t)row * gate_ld + h]) / sqrtf(ss / (float)d.vdim + d.eps);
#pragma unroll
    for (int c = 0; c < 4; ++c) {
        const int e = tid + 128 * c;
        if (e < d.vdim_p) out[((size_t)row * d.heads + h) * d.vdim_p + e] = __float2bfloat16_rn(acc[c] * f);
    }
}

typedef CUresult (*EncodeTiledFn)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *, const cuuint64_t *,
                                  const cuuint64_t *, const cuuint32_t *, const cuuint32_t *, CUtensorMapInterleave,
                                  CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

int columns_of(const DiffDims &d) { return d.group() <= 8 ? 16 : 32; }
int key_boxes(const DiffDims &d) { return (2 * d.dim_p + 63) / 64; }
int value_boxes(const DiffDims &d) { return 2 * ((d.vdim_p + 127) / 128); }
size_t stage_size(const DiffDims &d) { return (size_t)(key_boxes(d) + value_boxes(d)) * BOX; }
size_t fixed_smem(const DiffDims &d, int n) { return 1024 + (size_t)key_boxes(d) * n * 128 + (size_t)n * 512; }
constexpr size_t SMEM_MAX = 227 * 1024 - 2048;
int stages_of(const DiffDims &d) {
    const size_t fixed = fixed_smem(d, columns_of(d)), stage = stage_size(d);
    if (fixed + 2 * stage <= 111 * 1024) return 2; // two blocks per SM
    return fixed > SMEM_MAX ? 0 : (int)std::min<size_t>(3, (SMEM_MAX - fixed) / stage);
}
size_t smem_of(const DiffDims &d) { return fixed_smem(d, columns_of(d)) + stages_of(d) * stage_size(d); }

// Key splits per row: the number that minimises (waves of blocks) x (tiles per block + start-up).
int pick_splits(const b200nn_ctx *ctx, const DiffDims &d, int n_rows, int cap) {
    const int nh = columns_of(d) / 2, hb = d.kv_heads * ((d.group() + nh - 1) / nh), tiles = (cap + 127) / 128;
    const long long per_wave = (long long)ctx->sm_count * std::max<size_t>(1, (227 * 1024) / (smem_of(d) + 2048));
    int best = 1;
    double best_cost = 1e300;
    for (int s = 1; s <= std::min(tiles, 64); ++s) {
        const int per = (tiles + s - 1) / s;
        if (s > 1 && (tiles + s - 2) / (s - 1) == per) continue; // no shorter than with fewer splits
        const double waves = (double)(((long long)n_rows * hb * s + per_wave - 1) / per_wave);
        const double cost = waves * (per + 1.0);
        if (cost < best_cost) best_cost = cost, best = s;
    }
    return best;
}

template <int N>
int launch_n(b200nn_ctx *ctx, const DiffDecodeArgs &a, const CUtensorMap &tcm, int n_rows) {
    auto kern = diff_decode_tc_kernel<N>;
    static bool attr_done[16] = {};
    if (!attr_done[ctx->device & 15]) {
        CK(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM_MAX));
        prefer_max_smem(kern);
        attr_done[ctx->device & 15] = true;
    }
    const int nh = N / 2, blocks = a.d.kv_heads * ((a.d.group() + nh - 1) / nh);
    CK(ctx, launch_pdl(ctx, kern, dim3(a.splits, blocks, n_rows), dim3(NTHREADS), smem_of(a.d), tcm, a));
    CK_LAUNCH(ctx, "diff_decode_tc_kernel");
    return B200NN_OK;
}

}  // namespace

bool diff_decode_tc_supported(const b200nn_ctx *ctx, const DiffDims &d) {
    return ctx->attn_tc && ctx->encode_tiled && d.vdim_p <= 512 && columns_of(d) * (2 + value_boxes(d) / 2) <= 256 && stages_of(d) >= 1;
}

size_t diff_decode_tc_part_floats(const b200nn_ctx *ctx, const DiffDims &d, int n_rows, int cap) {
    return (size_t)pick_splits(ctx, d, n_rows, cap) * n_rows * d.heads * 2 * (d.vdim_p + 2);
}

int launch_diff_decode_tc(b200nn_ctx *ctx, const DiffDims &d, const __nv_bfloat16 *q, int ldq, const __nv_bfloat16 *cache, int cap, size_t cache_rows,
                          const RowMap &rows, int n_rows, const float *gate, int gate_ld, float *part, __nv_bfloat16 *out) {
    if (n_rows > 65535) return set_error(ctx, B200NN_ERR_SHAPE, "differential attention: more than 65535 rows");
    if (cache_rows > 0x7fffffff) return set_error(ctx, B200NN_ERR_SHAPE, "differential attention: more than 2^31 cache rows");
    DiffDecodeArgs a;
    a.d = d;
    a.rows = rows;
    a.q = q;
    a.ldq = ldq;
    a.cap = cap;
    a.splits = pick_splits(ctx, d, n_rows, cap);
    a.stages = stages_of(d);
    a.kb = key_boxes(d);
    a.vb = value_boxes(d);
    a.part_o = part;
    a.part_ml = part + (size_t)a.splits * n_rows * d.heads * 2 * d.vdim_p;
    a.dev_err = ctx->dev_err;
    CUtensorMap tcm;
    const cuuint64_t dim[2] = {(cuuint64_t)d.kv_w(), (cuuint64_t)cache_rows}, stride[1] = {(cuuint64_t)d.kv_w() * 2};
    const cuuint32_t box[2] = {64, 128}, ones[2] = {1, 1};
    CUresult r = ((EncodeTiledFn)ctx->encode_tiled)(&tcm, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, (void *)cache, dim, stride, box, ones,
                                                    CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
                                                    CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) return set_error(ctx, B200NN_ERR_CUDA, "cuTensorMapEncodeTiled (differential decode) failed: " + std::to_string((int)r));
    TRY(columns_of(d) == 16 ? launch_n<16>(ctx, a, tcm, n_rows) : launch_n<32>(ctx, a, tcm, n_rows));
    PREFER_SMEM_ONCE(diff_merge_kernel);
    CK(ctx, launch_pdl(ctx, diff_merge_kernel, dim3(d.heads, n_rows), dim3(128), 0, d, a.part_o, a.part_ml, a.splits, gate, gate_ld, out));
    CK_LAUNCH(ctx, "diff_merge_kernel");
    return B200NN_OK;
}
