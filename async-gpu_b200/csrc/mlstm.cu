// Matrix memory with exponential gates (mLSTM): a linear-attention recurrence whose state per head and sequence is one
// [dim, vdim] f32 matrix S, a normaliser n [dim] and a running maximum m.  With the log gates i = cap tanh(./cap) and
// f = logsigmoid(cap tanh(./cap)), per token
//     m' = max(f + m, i),  S' = e^(f + m - m') S + e^(i - m') k v^T,  n' the same with k alone,
//     o  = S'^T q / (max(|n' . q|, e^(-m')) + 1e-6),  q scaled by dim^(-1/2).
// Then o over its root mean square, times the norm weight, times sigmoid of the gate.  Everything here is f32.
//
//   mlstm_step_kernel   decoding: gates, recurrence, read-out, output norm and gate of one token
//   mlstm_gate_kernel   prompts: running maxima as a max-plus scan -> keep, write and floor e^(-m) of every row
//   mlstm_scan_kernel   prompts: the recurrence (state columns are independent; the normaliser is one more column,
//                       whose value is 1)
//   mlstm_out_kernel    prompts: division, output norm and gate
#include <algorithm>

#include "device_utils.cuh"
#include "hybrid.h"

namespace {

__device__ __forceinline__ float soft_cap(float v, float cap) { return cap * tanhf(v / cap); }
__device__ __forceinline__ float log_sigmoid_f(float v) { return fminf(v, 0.0f) - log1pf(expf(-fabsf(v))); }

// output gate (not part of the recurrence): fast exponential and division
__device__ __forceinline__ float gate_f(float v) { return __fdividef(1.0f, 1.0f + __expf(-v)); }

// ---- decoding ----------------------------------------------------------------------------------------
// Block = (row, head), eight warps; warp w holds state rows w, w + 8, ..., lane l columns 4l .. 4l+3 of a 128-column
// chunk.  Under the state's loads the threads fetch q, k, v, the gates and their entry of the normaliser.
template <int RPW, typename T>
__global__ void __launch_bounds__(256, RPW <= 16 ? 2 : 1)
mlstm_step_kernel(MlstmDims d, const float *__restrict__ proj, int ldp, MlstmWeights w, MlstmState state, RowMap rows, T *__restrict__ out) {
    extern __shared__ __align__(16) float sh[]; // q, k [dim_p], v, o [vdim_p], reduction [8][128], scalars [16]
    const int h = blockIdx.x, row = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    float *sq = sh, *sk = sq + d.dim_p, *sv = sk + d.dim_p, *so = sv + d.vdim_p, *red = so + d.vdim_p, *sc = red + 1024;
    pdl_trigger();
    pdl_wait();
    const int pos = row_pos(rows, row), slot = row_slot(rows, row);
    const size_t unit = (size_t)slot * d.heads + h;
    float *S = state.memory + unit * d.dim_p * d.vdim_p;
    float4 st[RPW];
    auto load_chunk = [&](int c0) {
        const bool col = c0 + lane * 4 < d.vdim_p;
#pragma unroll
        for (int r = 0; r < RPW; ++r) {
            const int i = warp + 8 * r;
            st[r] = col && i < d.dim_p && pos > 0 ? *reinterpret_cast<const float4 *>(S + (size_t)i * d.vdim_p + c0 + lane * 4)
                                                  : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    };
    load_chunk(0);
    const float *p = proj + (size_t)row * ldp;
    float ni = 0.0f, qi = 0.0f, ki = 0.0f; // this thread's entry of the normaliser (dim <= 256)
    if (tid < d.dim_p) {
        qi = p[d.q_at() + h * d.dim_p + tid] / sqrtf((float)d.dim);
        ki = p[d.k_at() + h * d.dim_p + tid];
        if (pos > 0) ni = state.normaliser[unit * d.dim_p + tid];
        sq[tid] = qi;
        sk[tid] = ki;
    }
    for (int j = tid; j < d.vdim_p; j += 256) sv[j] = p[d.v_at() + h * d.vdim_p + j];
    if (tid == 255) {
        const float i = soft_cap(p[d.i_at() + h] + w.i_bias[h], d.cap), f = log_sigmoid_f(soft_cap(p[d.f_at() + h] + w.f_bias[h], d.cap));
        const float m0 = pos > 0 ? state.maximum[unit] : 0.0f, m = fmaxf(f + m0, i);
        state.maximum[unit] = m;
        sc[0] = expf(f + m0 - m);
        sc[1] = expf(i - m);
        sc[2] = expf(-m);
    }
    __syncthreads();
    const float keep = sc[0], write = sc[1];
    ni = fmaf(keep, ni, write * ki);
    if (tid < d.dim_p) state.normaliser[unit * d.dim_p + tid] = ni;
    const float nq_part = warp_sum(ni * qi);
    if (lane == 0) sc[4 + warp] = nq_part;
    for (int c0 = 0; c0 < d.vdim_p; c0 += 128) {
        if (c0) load_chunk(c0);
        const int c = c0 + lane * 4;
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < d.vdim_p) {
            const float4 v = *reinterpret_cast<const float4 *>(sv + c);
            const float4 wv = make_float4(write * v.x, write * v.y, write * v.z, write * v.w);
#pragma unroll
            for (int r = 0; r < RPW; ++r) {
                const int i = warp + 8 * r;
                if (i < d.dim_p) {
                    const float k = sk[i], q = sq[i];
                    const float4 n = make_float4(fmaf(k, wv.x, keep * st[r].x), fmaf(k, wv.y, keep * st[r].y), fmaf(k, wv.z, keep * st[r].z),
                                                 fmaf(k, wv.w, keep * st[r].w));
                    *reinterpret_cast<float4 *>(S + (size_t)i * d.vdim_p + c) = n;
                    acc.x = fmaf(n.x, q, acc.x); acc.y = fmaf(n.y, q, acc.y); acc.z = fmaf(n.z, q, acc.z); acc.w = fmaf(n.w, q, acc.w);
                }
            }
        }
        *reinterpret_cast<float4 *>(red + warp * 128 + lane * 4) = acc;
        __syncthreads();
        if (warp == 0 && c < d.vdim_p) {
            float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int i = 0; i < 8; ++i) t = f4_add(t, *reinterpret_cast<const float4 *>(red + i * 128 + lane * 4));
            *reinterpret_cast<float4 *>(so + c) = t;
        }
        if (c0 + 128 < d.vdim_p) __syncthreads(); // red is used again
    }
    if (warp) return; // the read-out is warp 0's own
    __syncwarp();
    float nq = 0.0f;
#pragma unroll
    for (int i = 0; i < 8; ++i) nq += sc[4 + i];
    const float inv = 1.0f / (fmaxf(fabsf(nq), sc[2]) + 1e-6f);
    float s = 0.0f;
    for (int j = lane; j < d.vdim; j += 32) {
        const float o = so[j] * inv;
        s = fmaf(o, o, s);
    }
    const float rn = inv / sqrtf(warp_sum(s) / (float)d.vdim + d.eps);
    for (int j = lane; j < d.vdim; j += 32)
        store_from_float(out + ((size_t)row * d.heads + h) * d.vdim_p + j,
                         so[j] * rn * w.norm[h * d.vdim_p + j] * gate_f(p[d.g_at() + h * d.vdim_p + j]));
}

// ---- prompts -----------------------------------------------------------------------------------------
// Block = (head, sequence), eight warps, each with a contiguous segment of the tokens.  A token maps m to max(f + m, i); maps
// compose as (f1 + f2, max(i1 + f2, i2)), so 32 tokens are one warp scan and a segment is one map: the first pass over the
// tokens makes the segments' maps, the second starts from the maximum that enters its segment.  gates [row][head]: keep
// e^(f + m - m'), write e^(i - m'), floor e^(-m'), and room for n . q.
__global__ void __launch_bounds__(256)
mlstm_gate_kernel(MlstmDims d, const float *__restrict__ proj, int ldp, MlstmWeights w, MlstmState state, SeqMap sm, float4 *__restrict__ gates) {
    __shared__ float2 seg[8];
    const int h = blockIdx.x, sidx = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    pdl_trigger();
    const float ib = w.i_bias[h], fb = w.f_bias[h];
    pdl_wait();
    const int n = sm.n[sidx], row0 = sm.row0[sidx], per = (n + 255) / 256 * 32, t_beg = warp * per, t_end = min(n, t_beg + per);
    float *mp = state.maximum + (size_t)sm.slot[sidx] * d.heads + h;
    float m = sm.past[sidx] > 0 ? *mp : 0.0f;
    float i = 0.0f, f = 0.0f, a, b;
    auto scan = [&](int t) { // the lane's gates and the map from the group's start through its token; past the end the map is the identity
        const float *p = proj + (size_t)(row0 + min(t, n - 1)) * ldp;
        i = soft_cap(p[d.i_at() + h] + ib, d.cap);
        f = log_sigmoid_f(soft_cap(p[d.f_at() + h] + fb, d.cap));
        a = t < t_end ? f : 0.0f;
        b = t < t_end ? i : -INFINITY;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float pa = __shfl_up_sync(0xffffffffu, a, o), pb = __shfl_up_sync(0xffffffffu, b, o);
            if (lane >= o) {
                b = fmaxf(pb + a, b);
                a += pa;
            }
        }
    };
    float sa = 0.0f, sb = -INFINITY;
    for (int t0 = t_beg; t0 < t_end; t0 += 32) {
        scan(t0 + lane);
        const float ga = __shfl_sync(0xffffffffu, a, 31), gb = __shfl_sync(0xffffffffu, b, 31);
        sb = fmaxf(sb + ga, gb);
        sa += ga;
    }
    if (lane == 0) seg[warp] = make_float2(sa, sb);
    __syncthreads(); // every warp has also read the maximum the sequence came with
    for (int s = 0; s < warp; ++s) m = fmaxf(seg[s].x + m, seg[s].y);
    for (int t0 = t_beg; t0 < t_end; t0 += 32) {
        scan(t0 + lane);
        const float m_new = fmaxf(a + m, b);
        float m_old = __shfl_up_sync(0xffffffffu, m_new, 1);
        if (lane == 0) m_old = m;
        // from the maxima as they were rounded, so that their errors cancel along the sequence
        if (t0 + lane < t_end)
            gates[(size_t)(row0 + t0 + lane) * d.heads + h] = make_float4(expf(f + m_old - m_new), expf(i - m_new), expf(-m_new), 0.0f);
        m = __shfl_sync(0xffffffffu, m_new, 31);
    }
    if (lane == 0 && t_end == n && t_beg < n) *mp = m;
}

// Block = (16 NC state columns, head, sequence), four warps; the eight lanes of a column group hold its dim entries
// 4 l + 32 m .. + 3 of NC columns each (f32 pairs along dim).  Tokens come through shared memory TOK at a time, the next
// TOK being copied under the current ones.  The state is held divided by the decay G accumulated since it was last
// rescaled, so that a token costs two multiply-adds per entry.  The last block in x is the normaliser's: one column of
// warp 0, with value 1.
template <int DM, int NC>
__global__ void __launch_bounds__(128, DM > 4 ? 2 : 5)
mlstm_scan_kernel(MlstmDims d, const float *__restrict__ proj, int ldp, MlstmState state, SeqMap sm, float4 *__restrict__ gates,
                  float *__restrict__ heads_out) {
    constexpr int TOK = DM <= 4 ? 16 : 8, DP = DM * 32, CB = 16 * NC;
    struct Stage {
        float k[TOK][DP], q[TOK][DP], v[TOK][CB], s[TOK][4]; // s: keep, write
    };
    extern __shared__ __align__(16) uint8_t smem_raw[];
    Stage *stages = reinterpret_cast<Stage *>(smem_raw);
    pdl_trigger();
    const int cg = blockIdx.x, h = blockIdx.y, sidx = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const bool norm = cg == (int)gridDim.x - 1;
    const int part = lane & 7, cl = (warp * 4 + (lane >> 3)) * NC, col = norm ? cl : cg * CB + cl; // NC columns from col on
    const int cols = norm ? 1 : d.vdim_p;
    for (int i = tid; i < (int)(2 * sizeof(Stage) / 4); i += 128) reinterpret_cast<float *>(smem_raw)[i] = 0.0f; // entries past dim stay zero
    __syncthreads();
    if (norm && tid < 2 * TOK) stages[tid / TOK].v[tid % TOK][0] = 1.0f;
    pdl_wait();
    const int n = sm.n[sidx], past = sm.past[sidx], slot = sm.slot[sidx], row0 = sm.row0[sidx];
    const size_t unit = (size_t)slot * d.heads + h;
    float *S = norm ? state.normaliser + unit * d.dim_p : state.memory + unit * d.dim_p * d.vdim_p;
    uint64_t s[NC][DM * 2];
#pragma unroll
    for (int m = 0; m < DM; ++m)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
            const int i = 32 * m + 4 * part + e;
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                const bool in = i < d.dim_p && past > 0 && col + c < cols;
                s[c][2 * m + e / 2] = in ? f32x2(S[(size_t)i * cols + col + c], S[(size_t)(i + 1) * cols + col + c]) : 0ull;
            }
        }
    auto copy = [&](int t0, Stage &st) {
        const int nt = min(TOK, n - t0), cv = norm ? 0 : min(CB, d.vdim_p - cg * CB);
        for (int t = warp; t < nt; t += 4) { // a warp per token
            const float *c = proj + (size_t)(row0 + t0 + t) * ldp;
#pragma unroll
            for (int j = lane * 4; j < DP; j += 128)
                if (j < d.dim_p) {
                    cp_async16(&st.q[t][j], c + d.q_at() + h * d.dim_p + j);
                    cp_async16(&st.k[t][j], c + d.k_at() + h * d.dim_p + j);
                }
            if (lane * 4 < cv) cp_async16(&st.v[t][lane * 4], c + d.v_at() + h * d.vdim_p + cg * CB + lane * 4);
        }
        if (tid < nt) { // keep and write only: the other half of the row is being written by the normaliser's block
            const float *g = reinterpret_cast<const float *>(gates + (size_t)(row0 + t0 + tid) * d.heads + h);
            cp_async4(&st.s[tid][0], g);
            cp_async4(&st.s[tid][1], g + 1);
        }
    };
    copy(0, stages[0]);
    asm volatile("cp.async.commit_group;" ::: "memory");
    const float q_scale = 1.0f / sqrtf((float)d.dim);
    float G = 1.0f;
    auto rescale = [&](float f) {
        const uint64_t f2 = f32x2(f, f);
#pragma unroll
        for (int c = 0; c < NC; ++c)
#pragma unroll
            for (int m = 0; m < DM * 2; ++m) s[c][m] = mul2(f2, s[c][m]);
    };
    for (int t0 = 0, b = 0; t0 < n; t0 += TOK, b ^= 1) {
        if (t0 + TOK < n) copy(t0 + TOK, stages[b ^ 1]);
        asm volatile("cp.async.commit_group;" ::: "memory");
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();
        const Stage &st = stages[b];
        const int nt = norm && warp ? 0 : min(TOK, n - t0);
#pragma unroll 1
        for (int t = 0; t < nt; t += 4) { // four tokens' read-outs are reduced over the lanes together
            float r[4 * NC], g[4];        // partial sums of this lane, token by token; decay scale of each token
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const bool valid = t + x < nt;
                const float2 sc = *reinterpret_cast<const float2 *>(st.s[t + x]);
                G *= valid ? sc.x : 1.0f;
                if (G < 9.5367431640625e-7f) { // the same in every thread of the block
                    rescale(G);
                    G = 1.0f;
                }
                g[x] = G;
                const float wg = valid ? __fdividef(sc.y, G) : 0.0f;
                uint64_t u[NC], aq[NC];
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    const float y = wg * st.v[t + x][cl + c];
                    u[c] = f32x2(y, y);
                    aq[c] = 0ull;
                }
#pragma unroll
                for (int m = 0; m < DM; ++m) {
                    const ulonglong2 kk = *reinterpret_cast<const ulonglong2 *>(&st.k[t + x][32 * m + 4 * part]);
                    const ulonglong2 qq = *reinterpret_cast<const ulonglong2 *>(&st.q[t + x][32 * m + 4 * part]);
#pragma unroll
                    for (int c = 0; c < NC; ++c) {
                        s[c][2 * m] = fma2(kk.x, u[c], s[c][2 * m]);
                        s[c][2 * m + 1] = fma2(kk.y, u[c], s[c][2 * m + 1]);
                        aq[c] = fma2(s[c][2 * m], qq.x, aq[c]);
                        aq[c] = fma2(s[c][2 * m + 1], qq.y, aq[c]);
                    }
                }
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    const float2 p2 = f32x2_parts(aq[c]);
                    r[x * NC + c] = p2.x + p2.y;
                }
            }
            // transposing reduction over the eight lanes: value i of 4 NC ends in lane i (NC = 2) or lanes 2i, 2i + 1
            int o = 4;
#pragma unroll
            for (int k = 2 * NC; k >= 1; k >>= 1, o >>= 1) {
                const bool up = (lane & o) != 0;
#pragma unroll
                for (int i = 0; i < k; ++i) {
                    const float send = up ? r[i] : r[i + k], keep = up ? r[i + k] : r[i];
                    r[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
                }
            }
            if (NC == 1) r[0] += __shfl_xor_sync(0xffffffffu, r[0], 1);
            const int x = part >> 1, c = NC == 2 ? part & 1 : 0;
            const float v = (x < 2 ? (x == 0 ? g[0] : g[1]) : (x == 2 ? g[2] : g[3])) * q_scale * r[0];
            if (t + x < nt && (NC == 2 || !(part & 1)) && col + c < cols) {
                const size_t at = (size_t)(row0 + t0 + t + x) * d.heads + h;
                float *dst = norm ? &gates[at].w : heads_out + at * d.vdim_p + col + c;
                *dst = v;
            }
        }
        __syncthreads();
    }
    rescale(G);
#pragma unroll
    for (int m = 0; m < DM; ++m)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
            const int i = 32 * m + 4 * part + e;
#pragma unroll
            for (int c = 0; c < NC; ++c)
                if (i < d.dim_p && col + c < cols) {
                    const float2 v = f32x2_parts(s[c][2 * m + e / 2]);
                    S[(size_t)i * cols + col + c] = v.x;
                    S[(size_t)(i + 1) * cols + col + c] = v.y;
                }
        }
}

// One warp per (row, head).
template <typename T>
__global__ void __launch_bounds__(256)
mlstm_out_kernel(MlstmDims d, const float *__restrict__ proj, int ldp, const float *__restrict__ norm, const float4 *__restrict__ gates,
                 const float *__restrict__ heads_out, int n_rows, T *__restrict__ out) {
    pdl_trigger();
    pdl_wait();
    const int unit = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (unit >= n_rows * d.heads) return;
    const int row = unit / d.heads, h = unit - row * d.heads;
    const float *o = heads_out + (size_t)unit * d.vdim_p, *g = proj + (size_t)row * ldp + d.g_at() + h * d.vdim_p;
    const float4 gt = gates[unit];
    const float inv = 1.0f / (fmaxf(fabsf(gt.w), gt.z) + 1e-6f);
    float4 v[2]; // the first 256 columns stay in registers
    float s = 0.0f;
#pragma unroll
    for (int c = 0; c < 2; ++c) { // columns past vdim hold zeros
        const int j = lane * 4 + 128 * c;
        v[c] = j < d.vdim_p ? __ldcs(reinterpret_cast<const float4 *>(o + j)) : make_float4(0.f, 0.f, 0.f, 0.f);
        v[c].x *= inv; v[c].y *= inv; v[c].z *= inv; v[c].w *= inv;
        s += (v[c].x * v[c].x + v[c].y * v[c].y) + (v[c].z * v[c].z + v[c].w * v[c].w);
    }
    for (int j = 256 + lane; j < d.vdim_p; j += 32) s = fmaf(o[j] * inv, o[j] * inv, s);
    const float rn = 1.0f / sqrtf(warp_sum(s) / (float)d.vdim + d.eps);
    const float *nw = norm + h * d.vdim_p; // zero past vdim
    T *y = out + (size_t)unit * d.vdim_p;
#pragma unroll
    for (int c = 0; c < 2; ++c) {
        const int j = lane * 4 + 128 * c;
        if (j >= d.vdim_p) continue;
        const float4 gg = __ldcs(reinterpret_cast<const float4 *>(g + j)), ww = __ldg(reinterpret_cast<const float4 *>(nw + j));
        store_from_float(y + j, v[c].x * rn * ww.x * gate_f(gg.x));
        store_from_float(y + j + 1, v[c].y * rn * ww.y * gate_f(gg.y));
        store_from_float(y + j + 2, v[c].z * rn * ww.z * gate_f(gg.z));
        store_from_float(y + j + 3, v[c].w * rn * ww.w * gate_f(gg.w));
    }
    for (int j = 256 + lane; j < d.vdim_p; j += 32) store_from_float(y + j, o[j] * inv * rn * nw[j] * gate_f(g[j]));
}

template <typename T>
int step_launch(b200nn_ctx *ctx, const MlstmDims &d, const float *proj, int ldp, const MlstmWeights &w, const MlstmState &st, const RowMap &rows,
                int n_rows, T *out) {
    const dim3 grid(d.heads, n_rows);
    const size_t smem = (2 * d.dim_p + 2 * d.vdim_p + 1024 + 16) * sizeof(float);
#define MSTEP(R)                                                                                                      \
    do {                                                                                                              \
        PREFER_SMEM_ONCE((mlstm_step_kernel<R, T>));                                                                  \
        launch_pdl(ctx, mlstm_step_kernel<R, T>, grid, dim3(256), smem, d, proj, ldp, w, st, rows, out);              \
    } while (0)
    if (d.dim_p <= 64) MSTEP(8);
    else if (d.dim_p <= 128) MSTEP(16);
    else MSTEP(32);
#undef MSTEP
    CK_LAUNCH(ctx, "mlstm_step_kernel");
    return B200NN_OK;
}

}  // namespace

int launch_mlstm_step(b200nn_ctx *ctx, const MlstmDims &d, bool b16, const float *proj, int ldp, const MlstmWeights &w, const MlstmState &st,
                      const RowMap &rows, int n_rows, void *out) {
    if (n_rows > 65535) return set_error(ctx, B200NN_ERR_SHAPE, "mlstm: more than 65535 rows");
    if (d.dim_p > 256) return set_error(ctx, B200NN_ERR_UNSUPPORTED, "mlstm: dim > 256");
    return b16 ? step_launch(ctx, d, proj, ldp, w, st, rows, n_rows, (__nv_bfloat16 *)out)
               : step_launch(ctx, d, proj, ldp, w, st, rows, n_rows, (float *)out);
}

int launch_mlstm_prompt(b200nn_ctx *ctx, const MlstmDims &d, bool b16, const float *proj, int ldp, const MlstmWeights &w, const MlstmState &st,
                        const SeqMap &sm, int n_rows, float *gates, float *heads_out, void *out) {
    if (d.dim_p > 256) return set_error(ctx, B200NN_ERR_UNSUPPORTED, "mlstm: dim > 256");
    if (sm.n_seq > 65535) return set_error(ctx, B200NN_ERR_SHAPE, "mlstm: too many sequences in a pass");
    if (ldp & 3) return set_error(ctx, B200NN_ERR_SHAPE, "mlstm: projection rows must keep 16-byte alignment");
    PREFER_SMEM_ONCE(mlstm_gate_kernel);
    launch_pdl(ctx, mlstm_gate_kernel, dim3(d.heads, sm.n_seq), dim3(256), 0, d, proj, ldp, w, st, sm, (float4 *)gates);
    CK_LAUNCH(ctx, "mlstm_gate_kernel");
    // columns per lane: two when that leaves every SM a dozen warps, else one
    const long long columns = (long long)d.vdim_p * d.heads * sm.n_seq;
    const int dm = (d.dim_p + 31) / 32;
    const int nc = dm > 4 ? 1 : ctx->delta_cols ? ctx->delta_cols : columns >= 4LL * 2 * 10 * ctx->sm_count ? 2 : 1;
#define MSCAN(M, C)                                                                                                           \
    do {                                                                                                                      \
        constexpr int tok = M <= 4 ? 16 : 8;                                                                                  \
        constexpr size_t smem = 2 * sizeof(float) * tok * (2 * M * 32 + 16 * C + 4);                                          \
        static bool done[16] = {};                                                                                            \
        if (!done[ctx->device & 15]) {                                                                                        \
            CK(ctx, cudaFuncSetAttribute(mlstm_scan_kernel<M, C>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));   \
            prefer_max_smem(mlstm_scan_kernel<M, C>);                                                                         \
            done[ctx->device & 15] = true;                                                                                    \
        }                                                                                                                     \
        CK(ctx, launch_pdl(ctx, mlstm_scan_kernel<M, C>, dim3((d.vdim_p + 16 * C - 1) / (16 * C) + 1, d.heads, sm.n_seq),     \
                           dim3(128), smem, d, proj, ldp, st, sm, (float4 *)gates, heads_out));                               \
    } while (0)
#define MSCAN_C(M)                                                                                                            \
    do {                                                                                                                      \
        if (nc == 2) MSCAN(M, 2);                                                                                             \
        else MSCAN(M, 1);                                                                                                     \
    } while (0)
    if (dm <= 1) MSCAN_C(1);
    else if (dm <= 2) MSCAN_C(2);
    else if (dm <= 3) MSCAN_C(3);
    else if (dm <= 4) MSCAN_C(4);
    else if (dm <= 6) MSCAN(6, 1);
    else MSCAN(8, 1);
#undef MSCAN_C
#undef MSCAN
    CK_LAUNCH(ctx, "mlstm_scan_kernel");
    const int units = n_rows * d.heads;
    if (b16) {
        PREFER_SMEM_ONCE(mlstm_out_kernel<__nv_bfloat16>);
        launch_pdl(ctx, mlstm_out_kernel<__nv_bfloat16>, dim3((units + 7) / 8), dim3(256), 0, d, proj, ldp, w.norm, (const float4 *)gates, heads_out,
                   n_rows, (__nv_bfloat16 *)out);
    } else {
        PREFER_SMEM_ONCE(mlstm_out_kernel<float>);
        launch_pdl(ctx, mlstm_out_kernel<float>, dim3((units + 7) / 8), dim3(256), 0, d, proj, ldp, w.norm, (const float4 *)gates, heads_out, n_rows,
                   (float *)out);
    }
    CK_LAUNCH(ctx, "mlstm_out_kernel");
    return B200NN_OK;
}
