// Gated delta rule: a linear-attention recurrence whose state is one [dim, vdim] f32 matrix per head and
// sequence.  Per token S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q.  Both products against S are
// taken on the state before the write: S_new^T q = g S^T q + (k . q) u, so a token costs one pass over the
// state and one reduction instead of two.  Everything here is f32.
//
// The decay g is one number per head, or (CH, DeltaDims::channel) one per head and key channel, acting on the rows of
// S; the output gate is then a sigmoid and its input, like the decays', comes from a projection of its own (`ext`).
//
//   delta_step_kernel     decoding: convolution, norms, recurrence, output norm and gate of one token
//   delta_conv_kernel     prompts: convolution + silu, unit norms, k . q, decay and step size of every row
//   delta_scan_kernel     prompts: the recurrence (state columns are independent: a block owns some of them)
//   delta_out_kernel      prompts: output norm and gate
//
// The convolution's inputs are kept in a ring of `taps` rows per slot (position p in row p % taps): a token
// reads the other rows and replaces its own, so heads that share a query/key head do not race.
#include <algorithm>

#include "device_utils.cuh"
#include "hybrid.h"

namespace {

// activation of the convolution and of the output gate (not part of the recurrence): fast exponential and division
__device__ __forceinline__ float silu_f(float v) { return __fdividef(v, 1.0f + __expf(-v)); }
__device__ __forceinline__ float softplus_f(float v) { return v > 20.0f ? v : log1pf(expf(v)); }
__device__ __forceinline__ float decay_f(float a_exp, float a, float dt_bias) { return expf(-a_exp * softplus_f(a + dt_bias)); }

// ---- decoding ----------------------------------------------------------------------------------------
// Block = (row, head), eight warps.  Warp w holds state rows w, w + 8, ...; lane l columns 4l .. 4l+3 of a
// 128-column chunk (one chunk for vdim <= 128).  Under the state's loads warps 0, 1 and 2 make the query, key and value
// (a lane takes four channels; the unit norms stay scalar factors), warp 3 gate times norm weight, warp 4 decay and
// step size.
template <int RPW, bool CH, typename T>
__global__ void __launch_bounds__(256, RPW <= 16 ? 2 : 1)
delta_step_kernel(DeltaDims d, const float *__restrict__ proj, int ldp, const float *__restrict__ ext, DeltaWeights w, float *__restrict__ conv_state,
                  float *__restrict__ state, RowMap rows, T *__restrict__ out) {
    // q [dim_p], k [dim_p], v, gate, o [vdim_p], reduction [8][2][128], scalars [8], CH: decays [dim_p]
    extern __shared__ __align__(16) float sh[];
    const int h = blockIdx.x, row = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    float *sq = sh, *sk = sq + d.dim_p, *sv = sk + d.dim_p, *sgn = sv + d.vdim_p, *so = sgn + d.vdim_p, *red = so + d.vdim_p, *sc = red + 2048;
    float *sg = sc + 8;
    pdl_trigger();
    pdl_wait();
    const int pos = row_pos(rows, row), slot = row_slot(rows, row);
    float *S = state + ((size_t)slot * d.heads + h) * d.dim_p * d.vdim_p;
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
    const int group = d.heads / d.kv_heads, kh = h / group;
    const int cw = d.conv_w(), here = pos % d.taps;
    float *cring = conv_state + (size_t)slot * d.taps * cw;
    // four channels: the inputs of up to four taps are requested together, then summed; keep: put the input into the ring
    struct Taps {
        float4 x[4], w[4];
    };
    auto request = [&](int ch) {
        Taps t;
        t.x[0] = *reinterpret_cast<const float4 *>(p + ch);
        t.w[0] = __ldg(reinterpret_cast<const float4 *>(w.conv + (size_t)(d.taps - 1) * cw + ch));
#pragma unroll
        for (int i = 1; i < 4; ++i) {
            const bool use = i < d.taps && pos >= i;
            const int at = use ? (here - i < 0 ? here - i + d.taps : here - i) : here, tap = use ? d.taps - 1 - i : d.taps - 1;
            const float4 y = *reinterpret_cast<const float4 *>(cring + (size_t)at * cw + ch);
            t.x[i] = use ? y : make_float4(0.f, 0.f, 0.f, 0.f);
            t.w[i] = __ldg(reinterpret_cast<const float4 *>(w.conv + (size_t)tap * cw + ch));
        }
        return t;
    };
    auto channels = [&](const Taps &t, int ch, bool keep) {
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            a.x = fmaf(t.x[i].x, t.w[i].x, a.x); a.y = fmaf(t.x[i].y, t.w[i].y, a.y);
            a.z = fmaf(t.x[i].z, t.w[i].z, a.z); a.w = fmaf(t.x[i].w, t.w[i].w, a.w);
        }
        for (int i = 4; i < d.taps && pos >= i; ++i) {
            const float4 y = *reinterpret_cast<const float4 *>(cring + (size_t)(here - i < 0 ? here - i + d.taps : here - i) * cw + ch);
            const float4 wt = __ldg(reinterpret_cast<const float4 *>(w.conv + (size_t)(d.taps - 1 - i) * cw + ch));
            a.x = fmaf(y.x, wt.x, a.x); a.y = fmaf(y.y, wt.y, a.y); a.z = fmaf(y.z, wt.z, a.z); a.w = fmaf(y.w, wt.w, a.w);
        }
        if (keep) *reinterpret_cast<float4 *>(cring + (size_t)here * cw + ch) = t.x[0];
        return make_float4(silu_f(a.x), silu_f(a.y), silu_f(a.z), silu_f(a.w));
    };
    if (warp < 3) { // query, key, value
        const int n = warp < 2 ? d.dim_p : d.vdim_p, at = warp == 0 ? d.q_at() + kh * d.dim_p : warp == 1 ? d.k_at() + kh * d.dim_p : d.v_at() + h * d.vdim_p;
        float *dst = warp == 0 ? sq : warp == 1 ? sk : sv;
        float s = 0.0f;
        for (int j = lane * 4; j < n; j += 128) {
            const float4 a = channels(request(at + j), at + j, warp == 2 || h % group == 0);
            *reinterpret_cast<float4 *>(dst + j) = a;
            s += (a.x * a.x + a.y * a.y) + (a.z * a.z + a.w * a.w);
        }
        s = warp_sum(s);
        if (lane == 0) sc[2 + warp] = 1.0f / sqrtf(s + 1e-6f); // unit norms (the value's is not used)
    } else if (warp == 3) {
        for (int j = lane * 4; j < d.vdim_p; j += 128) { // the last columns may be padding: no norm weight there
            const float *gate = CH ? ext + (size_t)row * 2 * d.ext() + d.ext() : p + d.g_at();
            const float4 gg = *reinterpret_cast<const float4 *>(gate + h * d.vdim_p + j);
            const float e[4] = {gg.x, gg.y, gg.z, gg.w};
#pragma unroll
            for (int i = 0; i < 4; ++i) sgn[j + i] = j + i < d.vdim ? w.norm[j + i] * (CH ? sigmoid_f(e[i]) : silu_f(e[i])) : 0.0f;
        }
    } else if (CH && warp == 4) {
        if (lane == 0) sc[0] = sigmoid_f(p[d.b_at() + h]);
        const float a_exp = w.a_exp[h];
        for (int j = lane; j < d.dim_p; j += 32)
            sg[j] = decay_f(a_exp, ext[(size_t)row * 2 * d.ext() + h * d.dim_p + j], w.dt_bias[h * d.dim_p + j]);
    } else if (!CH && tid == 128) {
        sc[0] = sigmoid_f(p[d.b_at() + h]);
        sc[1] = decay_f(w.a_exp[h], p[d.a_at() + h], w.dt_bias[h]);
    }
    __syncthreads();
    const float beta = sc[0], g = CH ? 1.0f : sc[1], fq = sc[2] / sqrtf((float)d.dim), fk = sc[3]; // q also times dim^(-1/2)
    float kq = 0.0f; // warp 0, which makes the read-out, needs k . q
    if (warp == 0) {
        for (int j = lane; j < d.dim_p; j += 32) kq = fmaf(sk[j], sq[j], kq);
        kq = warp_sum(kq) * fq * fk;
    }
    for (int c0 = 0; c0 < d.vdim_p; c0 += 128) {
        if (c0) load_chunk(c0);
        float4 ak = make_float4(0.f, 0.f, 0.f, 0.f), aq = ak;
#pragma unroll
        for (int r = 0; r < RPW; ++r) {
            const int i = warp + 8 * r;
            if (i < d.dim_p) {
                const float gi = CH ? sg[i] : 1.0f, k = CH ? gi * sk[i] : sk[i], q = CH ? gi * sq[i] : sq[i];
                ak.x = fmaf(st[r].x, k, ak.x); ak.y = fmaf(st[r].y, k, ak.y); ak.z = fmaf(st[r].z, k, ak.z); ak.w = fmaf(st[r].w, k, ak.w);
                aq.x = fmaf(st[r].x, q, aq.x); aq.y = fmaf(st[r].y, q, aq.y); aq.z = fmaf(st[r].z, q, aq.z); aq.w = fmaf(st[r].w, q, aq.w);
            }
        }
        *reinterpret_cast<float4 *>(red + (warp * 2) * 128 + lane * 4) = ak;
        *reinterpret_cast<float4 *>(red + (warp * 2 + 1) * 128 + lane * 4) = aq;
        __syncthreads();
        float4 tk = make_float4(0.f, 0.f, 0.f, 0.f), tq = tk;
#pragma unroll
        for (int i = 0; i < 8; ++i) tk = f4_add(tk, *reinterpret_cast<const float4 *>(red + (i * 2) * 128 + lane * 4));
        if (warp == 0)
#pragma unroll
            for (int i = 0; i < 8; ++i) tq = f4_add(tq, *reinterpret_cast<const float4 *>(red + (i * 2 + 1) * 128 + lane * 4));
        const int c = c0 + lane * 4;
        if (c < d.vdim_p) {
            const float4 v = *reinterpret_cast<const float4 *>(sv + c);
            const float gk = g * fk, gq = g * fq;
            const float4 u = make_float4(beta * (v.x - gk * tk.x), beta * (v.y - gk * tk.y), beta * (v.z - gk * tk.z), beta * (v.w - gk * tk.w));
#pragma unroll
            for (int r = 0; r < RPW; ++r) {
                const int i = warp + 8 * r;
                if (i < d.dim_p) {
                    const float k = sk[i] * fk, gi = CH ? sg[i] : g;
                    *reinterpret_cast<float4 *>(S + (size_t)i * d.vdim_p + c) =
                        make_float4(fmaf(k, u.x, gi * st[r].x), fmaf(k, u.y, gi * st[r].y), fmaf(k, u.z, gi * st[r].z), fmaf(k, u.w, gi * st[r].w));
                }
            }
            if (warp == 0)
                *reinterpret_cast<float4 *>(so + c) =
                    make_float4(fmaf(kq, u.x, gq * tq.x), fmaf(kq, u.y, gq * tq.y), fmaf(kq, u.z, gq * tq.z), fmaf(kq, u.w, gq * tq.w));
        }
        if (c0 + 128 < d.vdim_p) __syncthreads(); // red is used again
    }
    if (warp) return; // the read-out is warp 0's own
    __syncwarp();
    float s = 0.0f;
    for (int j = lane; j < d.vdim; j += 32) s = fmaf(so[j], so[j], s);
    const float rn = 1.0f / sqrtf(warp_sum(s) / (float)d.vdim + d.eps);
    for (int j = lane; j < d.vdim; j += 32) store_from_float(out + ((size_t)row * d.heads + h) * d.vdim_p + j, so[j] * rn * sgn[j]);
}

// ---- prompts -----------------------------------------------------------------------------------------
// Columns of the convolved rows: q (scaled), k, v as in the projection, then per head the decay and the step size,
// then per query/key head k . q; rows DeltaDims::conv_ld() apart.
//
// A warp takes four rows of one unit: a query/key head (both of its vectors) or a value head.  The eight warps of a
// block take neighbouring rows, which share their convolution inputs in L1.
// NCH: 128-channel chunks of a query/key head.
constexpr int CONV_ROWS = 4;
template <int NCH, bool CH>
__global__ void __launch_bounds__(256)
delta_conv_kernel(DeltaDims d, const float *__restrict__ proj, int ldp, const float *__restrict__ ext, DeltaWeights w, const float *__restrict__ conv_state, RowMap rows,
                  SeqMap sm, const int *__restrict__ row_seq, int n_rows, float *__restrict__ conv) {
    pdl_trigger();
    pdl_wait();
    const int r_first = (blockIdx.y * 8 + (threadIdx.x >> 5)) * CONV_ROWS, u = blockIdx.x, lane = threadIdx.x & 31;
    const int cw = d.conv_w(), ld = d.conv_ld();
    int pos[CONV_ROWS], back[CONV_ROWS]; // position; rows of the same sequence before it in the pass
    const float *cring[CONV_ROWS];
#pragma unroll
    for (int r = 0; r < CONV_ROWS; ++r) {
        const int row = min(r_first + r, n_rows - 1);
        pos[r] = row_pos(rows, row);
        back[r] = row - sm.row0[row_seq[row]];
        cring[r] = conv_state + (size_t)row_slot(rows, row) * d.taps * cw;
    }
    // channels ch .. ch+3 of row r_first + r after convolution and silu
    auto channels = [&](int r, int ch) {
        const float *p = proj + (size_t)min(r_first + r, n_rows - 1) * ldp;
        const float4 x = *reinterpret_cast<const float4 *>(p + ch), w0 = __ldg(reinterpret_cast<const float4 *>(w.conv + (size_t)(d.taps - 1) * cw + ch));
        float4 a = make_float4(x.x * w0.x, x.y * w0.y, x.z * w0.z, x.w * w0.w);
        for (int t = 1; t < d.taps && pos[r] - t >= 0; ++t) {
            const float4 y = *reinterpret_cast<const float4 *>(back[r] >= t ? p - (size_t)t * ldp + ch : cring[r] + (size_t)((pos[r] - t) % d.taps) * cw + ch);
            const float4 wt = __ldg(reinterpret_cast<const float4 *>(w.conv + (size_t)(d.taps - 1 - t) * cw + ch));
            a.x = fmaf(y.x, wt.x, a.x); a.y = fmaf(y.y, wt.y, a.y); a.z = fmaf(y.z, wt.z, a.z); a.w = fmaf(y.w, wt.w, a.w);
        }
        return make_float4(silu_f(a.x), silu_f(a.y), silu_f(a.z), silu_f(a.w));
    };
    // the same for all four rows; four neighbours of one sequence with their inputs in the pass share seven loads
    const bool shared = d.taps <= 4 && back[0] >= 3 && back[CONV_ROWS - 1] == back[0] + CONV_ROWS - 1 && r_first + CONV_ROWS <= n_rows;
    auto rows4 = [&](int ch, float4 (&o)[CONV_ROWS]) {
        if (!shared) {
#pragma unroll
            for (int r = 0; r < CONV_ROWS; ++r) o[r] = channels(r, ch);
            return;
        }
        float4 x[CONV_ROWS + 3], wt[4];
#pragma unroll
        for (int i = 0; i < CONV_ROWS + 3; ++i) x[i] = *reinterpret_cast<const float4 *>(proj + (size_t)(r_first + i - 3) * ldp + ch);
#pragma unroll
        for (int t = 0; t < 4; ++t)
            wt[t] = t < d.taps ? __ldg(reinterpret_cast<const float4 *>(w.conv + (size_t)(d.taps - 1 - t) * cw + ch)) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int r = 0; r < CONV_ROWS; ++r) {
            float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int t = 0; t < 4; ++t) {
                const float4 y = x[3 + r - t];
                a.x = fmaf(y.x, wt[t].x, a.x); a.y = fmaf(y.y, wt[t].y, a.y); a.z = fmaf(y.z, wt[t].z, a.z); a.w = fmaf(y.w, wt[t].w, a.w);
            }
            o[r] = make_float4(silu_f(a.x), silu_f(a.y), silu_f(a.z), silu_f(a.w));
        }
    };
    if (u >= d.kv_heads) { // a value head
        const int h = u - d.kv_heads;
        for (int j = lane * 4; j < d.vdim_p; j += 128) {
            float4 v[CONV_ROWS];
            rows4(d.v_at() + h * d.vdim_p + j, v);
#pragma unroll
            for (int r = 0; r < CONV_ROWS; ++r)
                if (r_first + r < n_rows) *reinterpret_cast<float4 *>(conv + (size_t)(r_first + r) * ld + d.v_at() + h * d.vdim_p + j) = v[r];
        }
        if (lane < CONV_ROWS && r_first + lane < n_rows) {
            const float *p = proj + (size_t)(r_first + lane) * ldp;
            float *o = conv + (size_t)(r_first + lane) * ld;
            if (!CH) o[d.decay_at() + h] = decay_f(w.a_exp[h], p[d.a_at() + h], w.dt_bias[h]);
            o[d.beta_at() + h] = sigmoid_f(p[d.b_at() + h]);
        }
        if (CH) {
            const float a_exp = w.a_exp[h];
            for (int j = lane * 4; j < d.dim_p; j += 128) {
                const float4 b = __ldg(reinterpret_cast<const float4 *>(w.dt_bias + h * d.dim_p + j));
#pragma unroll
                for (int r = 0; r < CONV_ROWS; ++r) {
                    if (r_first + r >= n_rows) break;
                    const float4 a = *reinterpret_cast<const float4 *>(ext + (size_t)(r_first + r) * 2 * d.ext() + h * d.dim_p + j);
                    *reinterpret_cast<float4 *>(conv + (size_t)(r_first + r) * ld + d.decay_at() + h * d.dim_p + j) =
                        make_float4(decay_f(a_exp, a.x, b.x), decay_f(a_exp, a.y, b.y), decay_f(a_exp, a.z, b.z), decay_f(a_exp, a.w, b.w));
                }
            }
        }
        return;
    }
    const float q_scale = 1.0f / sqrtf((float)d.dim);
    float4 q[NCH][CONV_ROWS], k[NCH][CONV_ROWS];
#pragma unroll
    for (int c = 0; c < NCH; ++c) {
        const int j = lane * 4 + 128 * c;
#pragma unroll
        for (int r = 0; r < CONV_ROWS; ++r) q[c][r] = k[c][r] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (j < d.dim_p) {
            rows4(d.q_at() + u * d.dim_p + j, q[c]);
            rows4(d.k_at() + u * d.dim_p + j, k[c]);
        }
    }
#pragma unroll
    for (int r = 0; r < CONV_ROWS; ++r) {
        float qq = 0.0f, kk = 0.0f, kq = 0.0f;
#pragma unroll
        for (int c = 0; c < NCH; ++c) {
            const float4 a = q[c][r], b = k[c][r];
            qq += (a.x * a.x + a.y * a.y) + (a.z * a.z + a.w * a.w);
            kk += (b.x * b.x + b.y * b.y) + (b.z * b.z + b.w * b.w);
            kq += (a.x * b.x + a.y * b.y) + (a.z * b.z + a.w * b.w);
        }
        const float fq = q_scale / sqrtf(warp_sum(qq) + 1e-6f), fk = 1.0f / sqrtf(warp_sum(kk) + 1e-6f);
        const float dot = warp_sum(kq) * fq * fk;
        if (r_first + r >= n_rows) continue;
        float *o = conv + (size_t)(r_first + r) * ld;
#pragma unroll
        for (int c = 0; c < NCH; ++c) {
            const int j = lane * 4 + 128 * c;
            if (j < d.dim_p) {
                const float4 a = q[c][r], b = k[c][r];
                *reinterpret_cast<float4 *>(o + d.q_at() + u * d.dim_p + j) = make_float4(a.x * fq, a.y * fq, a.z * fq, a.w * fq);
                *reinterpret_cast<float4 *>(o + d.k_at() + u * d.dim_p + j) = make_float4(b.x * fk, b.y * fk, b.z * fk, b.w * fk);
            }
        }
        if (lane == 0) o[d.kq_at() + u] = dot;
    }
}

// Block = (16 NC state columns, head, sequence), four warps.  The eight lanes of a column group hold its dim entries
// 4 l + 32 m .. + 3 of NC columns each (f32 pairs along dim).  Tokens come through shared memory TOK at a time, the next
// TOK being copied under the current ones.  The state is held divided by the decay G accumulated since it was last
// rescaled (S = G s), so that a token costs three multiply-adds per entry; it is rescaled when G falls below 2^-20.
// With CH the decays differ along dim and are multiplied in directly (one multiply more per entry).
// Per token: both products against the old state, one reduction over the eight lanes (transposing: 2 NC values in
// log steps), the write.  Also leaves the convolution's last inputs in the cache (blocks of column group 0).
template <int DM, int NC, bool CH>
__global__ void __launch_bounds__(128, DM > 4 ? 1 : 4)
delta_scan_kernel(DeltaDims d, const float *__restrict__ proj, int ldp, const float *__restrict__ conv, float *__restrict__ conv_state,
                  float *__restrict__ state, SeqMap sm, float *__restrict__ heads_out) {
    constexpr int TOK = DM <= 4 ? 16 : 8, DP = DM * 32, CB = 16 * NC;
    struct Stage {
        float k[TOK][DP], q[TOK][DP], v[TOK][CB], s[TOK][4], g[CH ? TOK : 1][CH ? DP : 4]; // s: decay, step size, k . q; g: decays
    };
    extern __shared__ __align__(16) uint8_t smem_raw[];
    Stage *stages = reinterpret_cast<Stage *>(smem_raw);
    pdl_trigger();
    const int cg = blockIdx.x, h = blockIdx.y, sidx = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int part = lane & 7, cl = (warp * 4 + (lane >> 3)) * NC, col = cg * CB + cl; // NC columns from col on
    for (int i = tid; i < (int)(2 * sizeof(Stage) / 4); i += 128) reinterpret_cast<float *>(smem_raw)[i] = 0.0f; // entries past dim stay zero
    pdl_wait();
    const int n = sm.n[sidx], past = sm.past[sidx], slot = sm.slot[sidx], row0 = sm.row0[sidx];
    const int group = d.heads / d.kv_heads, kh = h / group, cw = d.conv_w(), ldc = d.conv_ld();
    float *S = state + ((size_t)slot * d.heads + h) * d.dim_p * d.vdim_p + col;
    uint64_t s[NC][DM * 2];
#pragma unroll
    for (int m = 0; m < DM; ++m)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
            const int i = 32 * m + 4 * part + e;
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                const bool in = i < d.dim_p && past > 0 && col + c < d.vdim_p;
                s[c][2 * m + e / 2] = in ? f32x2(S[(size_t)i * d.vdim_p + c], S[(size_t)(i + 1) * d.vdim_p + c]) : 0ull;
            }
        }
    auto copy = [&](int t0, Stage &st) {
        const int nt = min(TOK, n - t0), dv = d.dim_p >> 2, cv = min(CB, d.vdim_p - cg * CB) >> 2;
        const float *c = conv + (size_t)(row0 + t0) * ldc;
        for (int i = tid; i < nt * dv; i += 128) {
            const int t = i / dv, j = (i - t * dv) * 4;
            cp_async16(&st.q[t][j], c + (size_t)t * ldc + d.q_at() + kh * d.dim_p + j);
            cp_async16(&st.k[t][j], c + (size_t)t * ldc + d.k_at() + kh * d.dim_p + j);
            if constexpr (CH) cp_async16(&st.g[t][j], c + (size_t)t * ldc + d.decay_at() + h * d.dim_p + j);
        }
        for (int i = tid; i < nt * cv; i += 128) {
            const int t = i / cv, j = (i - t * cv) * 4;
            cp_async16(&st.v[t][j], c + (size_t)t * ldc + d.v_at() + h * d.vdim_p + cg * CB + j);
        }
        for (int i = tid; i < nt * 3; i += 128) {
            const int t = i / 3, j = i - t * 3;
            if (CH && j == 0) continue;
            cp_async4(&st.s[t][j], c + (size_t)t * ldc + (j == 0 ? d.decay_at() + h : j == 1 ? d.beta_at() + h : d.kq_at() + kh));
        }
    };
    __syncthreads();
    copy(0, stages[0]);
    asm volatile("cp.async.commit_group;" ::: "memory");
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
        const int nt = min(TOK, n - t0);
#pragma unroll 4
        for (int t = 0; t < nt; ++t) {
            const float4 sc = *reinterpret_cast<const float4 *>(st.s[t]);
            if constexpr (CH) {
#pragma unroll
                for (int m = 0; m < DM; ++m) {
                    const ulonglong2 gg = *reinterpret_cast<const ulonglong2 *>(&st.g[t][32 * m + 4 * part]);
#pragma unroll
                    for (int c = 0; c < NC; ++c) {
                        s[c][2 * m] = mul2(gg.x, s[c][2 * m]);
                        s[c][2 * m + 1] = mul2(gg.y, s[c][2 * m + 1]);
                    }
                }
            } else {
                G *= sc.x;
                if (G < 9.5367431640625e-7f) { // the same in every thread of the block
                    rescale(G);
                    G = 1.0f;
                }
            }
            uint64_t k[DM * 2];
            float r[2 * NC]; // s^T k of the NC columns, then s^T q
            {
                uint64_t ak[NC], aq[NC];
#pragma unroll
                for (int c = 0; c < NC; ++c) ak[c] = aq[c] = 0ull;
#pragma unroll
                for (int m = 0; m < DM; ++m) {
                    const ulonglong2 kk = *reinterpret_cast<const ulonglong2 *>(&st.k[t][32 * m + 4 * part]);
                    const ulonglong2 qq = *reinterpret_cast<const ulonglong2 *>(&st.q[t][32 * m + 4 * part]);
                    k[2 * m] = kk.x;
                    k[2 * m + 1] = kk.y;
#pragma unroll
                    for (int c = 0; c < NC; ++c) {
                        ak[c] = fma2(s[c][2 * m], kk.x, ak[c]);
                        aq[c] = fma2(s[c][2 * m], qq.x, aq[c]);
                        ak[c] = fma2(s[c][2 * m + 1], kk.y, ak[c]);
                        aq[c] = fma2(s[c][2 * m + 1], qq.y, aq[c]);
                    }
                }
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    const float2 a = f32x2_parts(ak[c]), q = f32x2_parts(aq[c]);
                    r[c] = a.x + a.y;
                    r[NC + c] = q.x + q.y;
                }
            }
            // reduction over the eight lanes of the group: halve the values while there are several, then plain
            int o = 4;
#pragma unroll
            for (int w = NC; w >= 1; w >>= 1, o >>= 1) {
                const bool up = (lane & o) != 0;
#pragma unroll
                for (int i = 0; i < w; ++i) {
                    const float send = up ? r[i] : r[i + w], keep = up ? r[i + w] : r[i];
                    r[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
                }
            }
            for (; o; o >>= 1) r[0] += __shfl_xor_sync(0xffffffffu, r[0], o);
            // lanes with bit 4 clear now hold s^T k, the others s^T q, of column idx
            const int idx = NC == 1 ? 0 : (lane >> 1) & 1;
            const float mine = CH ? r[0] : G * r[0], other = __shfl_xor_sync(0xffffffffu, mine, 4);
            const float u_own = sc.y * (st.v[t][cl + idx] - ((lane & 4) ? other : mine));
            if ((lane & 4) && !(lane & 1) && (NC == 2 || !(lane & 2)) && col + idx < d.vdim_p)
                heads_out[((size_t)(row0 + t0 + t) * d.heads + h) * d.vdim_p + col + idx] = fmaf(sc.z, u_own, mine);
            const float us = CH ? u_own : __fdividef(u_own, G);
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                const float u = NC == 1 ? us : __shfl_sync(0xffffffffu, us, (lane & 24) | (c << 1));
                const uint64_t u2 = f32x2(u, u);
#pragma unroll
                for (int m = 0; m < DM * 2; ++m) s[c][m] = fma2(k[m], u2, s[c][m]);
            }
        }
        __syncthreads();
    }
    if (!CH) rescale(G);
#pragma unroll
    for (int m = 0; m < DM; ++m)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
            const int i = 32 * m + 4 * part + e;
#pragma unroll
            for (int c = 0; c < NC; ++c)
                if (i < d.dim_p && col + c < d.vdim_p) {
                    const float2 v = f32x2_parts(s[c][2 * m + e / 2]);
                    S[(size_t)i * d.vdim_p + c] = v.x;
                    S[(size_t)(i + 1) * d.vdim_p + c] = v.y;
                }
        }
    if (cg == 0) {
        float *cring = conv_state + (size_t)slot * d.taps * cw;
        for (int t = max(0, n - d.taps); t < n; ++t) {
            const float *p = proj + (size_t)(row0 + t) * ldp;
            float *c = cring + (size_t)((past + t) % d.taps) * cw;
            if (h % group == 0)
                for (int j = tid; j < d.dim_p; j += 128) {
                    c[d.q_at() + kh * d.dim_p + j] = p[d.q_at() + kh * d.dim_p + j];
                    c[d.k_at() + kh * d.dim_p + j] = p[d.k_at() + kh * d.dim_p + j];
                }
            for (int j = tid; j < d.vdim_p; j += 128) c[d.v_at() + h * d.vdim_p + j] = p[d.v_at() + h * d.vdim_p + j];
        }
    }
}

// One warp per (row, head).
template <bool CH, typename T>
__global__ void __launch_bounds__(256)
delta_out_kernel(DeltaDims d, const float *__restrict__ gates, int ldg, const float *__restrict__ norm, const float *__restrict__ heads_out,
                 int n_rows, T *__restrict__ out) {
    pdl_trigger();
    pdl_wait();
    const int unit = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (unit >= n_rows * d.heads) return;
    const int row = unit / d.heads, h = unit - row * d.heads;
    const float *o = heads_out + (size_t)unit * d.vdim_p, *g = gates + (size_t)row * ldg + h * d.vdim_p;
    auto act = [](float z) { return CH ? sigmoid_f(z) : silu_f(z); };
    float4 v[2]; // the first 256 columns stay in registers
    float s = 0.0f;
#pragma unroll
    for (int c = 0; c < 2; ++c) { // columns past vdim hold zeros
        const int j = lane * 4 + 128 * c;
        v[c] = j < d.vdim_p ? __ldcs(reinterpret_cast<const float4 *>(o + j)) : make_float4(0.f, 0.f, 0.f, 0.f);
        s += (v[c].x * v[c].x + v[c].y * v[c].y) + (v[c].z * v[c].z + v[c].w * v[c].w);
    }
    for (int j = 256 + lane; j < d.vdim_p; j += 32) s = fmaf(o[j], o[j], s);
    const float rn = 1.0f / sqrtf(warp_sum(s) / (float)d.vdim + d.eps);
    T *y = out + (size_t)unit * d.vdim_p;
#pragma unroll
    for (int c = 0; c < 2; ++c) {
        const int j = lane * 4 + 128 * c;
        if (j >= d.vdim_p) continue;
        const float4 gg = __ldcs(reinterpret_cast<const float4 *>(g + j));
        const float e[4] = {v[c].x * act(gg.x), v[c].y * act(gg.y), v[c].z * act(gg.z), v[c].w * act(gg.w)};
#pragma unroll
        for (int i = 0; i < 4; ++i) store_from_float(y + j + i, j + i < d.vdim ? e[i] * rn * norm[j + i] : 0.0f);
    }
    for (int j = 256 + lane; j < d.vdim; j += 32) store_from_float(y + j, o[j] * rn * norm[j] * act(g[j]));
}

template <bool CH, typename T>
int step_launch(b200nn_ctx *ctx, const DeltaDims &d, const float *proj, int ldp, const float *ext, const DeltaWeights &w, float *conv_state, float *state,
                const RowMap &rows, int n_rows, T *out) {
    const dim3 grid(d.heads, n_rows);
    const size_t smem = (2 * d.dim_p + 3 * d.vdim_p + 2048 + 8 + (CH ? d.dim_p : 0)) * sizeof(float);
#define DSTEP(R)                                                                                                             \
    do {                                                                                                                     \
        PREFER_SMEM_ONCE((delta_step_kernel<R, CH, T>));                                                                     \
        launch_pdl(ctx, delta_step_kernel<R, CH, T>, grid, dim3(256), smem, d, proj, ldp, ext, w, conv_state, state, rows,   \
                   out);                                                                                                     \
    } while (0)
    if (d.dim_p <= 64) DSTEP(8);
    else if (d.dim_p <= 128) DSTEP(16);
    else DSTEP(32);
#undef DSTEP
    CK_LAUNCH(ctx, "delta_step_kernel");
    return B200NN_OK;
}

template <bool CH>
int prompt_launch(b200nn_ctx *ctx, const DeltaDims &d, bool b16, const float *proj, int ldp, const float *ext, const DeltaWeights &w, float *conv_state,
                  float *state, const RowMap &rows, const SeqMap &sm, int n_rows, const int *row_seq, float *conv, float *heads_out, void *out) {
    const dim3 cgrid(d.kv_heads + d.heads, (n_rows + 8 * CONV_ROWS - 1) / (8 * CONV_ROWS));
    PREFER_SMEM_ONCE((delta_conv_kernel<1, CH>));
    PREFER_SMEM_ONCE((delta_conv_kernel<2, CH>));
    if (d.dim_p <= 128)
        launch_pdl(ctx, delta_conv_kernel<1, CH>, cgrid, dim3(256), 0, d, proj, ldp, ext, w, conv_state, rows, sm, row_seq, n_rows, conv);
    else
        launch_pdl(ctx, delta_conv_kernel<2, CH>, cgrid, dim3(256), 0, d, proj, ldp, ext, w, conv_state, rows, sm, row_seq, n_rows, conv);
    CK_LAUNCH(ctx, "delta_conv_kernel");
    // columns per lane: two when that leaves every SM a dozen warps, else one (more parallel, more instructions)
    const long long columns = (long long)d.vdim_p * d.heads * sm.n_seq;
    const int dm = (d.dim_p + 31) / 32;
    const int nc = dm > 4 ? 1 : ctx->delta_cols ? ctx->delta_cols : columns >= 4LL * 2 * 10 * ctx->sm_count ? 2 : 1;
#define DSCAN(M, C)                                                                                                           \
    do {                                                                                                                      \
        constexpr int ch = M <= 4 ? 16 : 8;                                                                                   \
        constexpr size_t smem = 2 * sizeof(float) * (ch * (2 * M * 32 + 16 * C + 4) + (CH ? ch * M * 32 : 4));                \
        static bool done[16] = {};                                                                                            \
        if (!done[ctx->device & 15]) {                                                                                        \
            CK(ctx, cudaFuncSetAttribute(delta_scan_kernel<M, C, CH>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
            prefer_max_smem(delta_scan_kernel<M, C, CH>);                                                                     \
            done[ctx->device & 15] = true;                                                                                    \
        }                                                                                                                     \
        CK(ctx, launch_pdl(ctx, delta_scan_kernel<M, C, CH>, dim3((d.vdim_p + 16 * C - 1) / (16 * C), d.heads, sm.n_seq),     \
                           dim3(128), smem, d, proj, ldp, conv, conv_state, state, sm, heads_out));                           \
    } while (0)
#define DSCAN_C(M)                                                                                                            \
    do {                                                                                                                      \
        if (nc == 2) DSCAN(M, 2);                                                                                             \
        else DSCAN(M, 1);                                                                                                     \
    } while (0)
    if (dm <= 1) DSCAN_C(1);
    else if (dm <= 2) DSCAN_C(2);
    else if (dm <= 3) DSCAN_C(3);
    else if (dm <= 4) DSCAN_C(4);
    else if (dm <= 6) DSCAN(6, 1);
    else DSCAN(8, 1);
#undef DSCAN_C
#undef DSCAN
    CK_LAUNCH(ctx, "delta_scan_kernel");
    const int units = n_rows * d.heads;
    const float *gates = CH ? ext + d.ext() : proj + d.g_at();
    const int ldg = CH ? 2 * d.ext() : ldp;
    if (b16) {
        PREFER_SMEM_ONCE((delta_out_kernel<CH, __nv_bfloat16>));
        launch_pdl(ctx, delta_out_kernel<CH, __nv_bfloat16>, dim3((units + 7) / 8), dim3(256), 0, d, gates, ldg, w.norm, heads_out, n_rows,
                   (__nv_bfloat16 *)out);
    } else {
        PREFER_SMEM_ONCE((delta_out_kernel<CH, float>));
        launch_pdl(ctx, delta_out_kernel<CH, float>, dim3((units + 7) / 8), dim3(256), 0, d, gates, ldg, w.norm, heads_out, n_rows, (float *)out);
    }
    CK_LAUNCH(ctx, "delta_out_kernel");
    return B200NN_OK;
}

}  // namespace

int launch_delta_step(b200nn_ctx *ctx, const DeltaDims &d, bool b16, const float *proj, int ldp, const float *ext, const DeltaWeights &w, float *conv_state,
                      float *state, const RowMap &rows, int n_rows, void *out) {
    if (n_rows > 65535) return set_error(ctx, B200NN_ERR_SHAPE, "delta rule: more than 65535 rows");
    if (d.dim_p > 256) return set_error(ctx, B200NN_ERR_UNSUPPORTED, "delta rule: dim > 256");
    if (d.channel)
        return b16 ? step_launch<true>(ctx, d, proj, ldp, ext, w, conv_state, state, rows, n_rows, (__nv_bfloat16 *)out)
                   : step_launch<true>(ctx, d, proj, ldp, ext, w, conv_state, state, rows, n_rows, (float *)out);
    return b16 ? step_launch<false>(ctx, d, proj, ldp, ext, w, conv_state, state, rows, n_rows, (__nv_bfloat16 *)out)
               : step_launch<false>(ctx, d, proj, ldp, ext, w, conv_state, state, rows, n_rows, (float *)out);
}

int launch_delta_prompt(b200nn_ctx *ctx, const DeltaDims &d, bool b16, const float *proj, int ldp, const float *ext, const DeltaWeights &w,
                        float *conv_state, float *state, const RowMap &rows, const SeqMap &sm, int n_rows, const int *row_seq, float *conv,
                        float *heads_out, void *out) {
    if (d.dim_p > 256) return set_error(ctx, B200NN_ERR_UNSUPPORTED, "delta rule: dim > 256");
    if (n_rows > 8 * 65535 || sm.n_seq > 65535) return set_error(ctx, B200NN_ERR_SHAPE, "delta rule: too many rows or sequences in a pass");
    if (ldp & 3) return set_error(ctx, B200NN_ERR_SHAPE, "delta rule: projection rows must keep 16-byte alignment");
    return d.channel ? prompt_launch<true>(ctx, d, b16, proj, ldp, ext, w, conv_state, state, rows, sm, n_rows, row_seq, conv, heads_out, out)
                     : prompt_launch<false>(ctx, d, b16, proj, ldp, ext, w, conv_state, state, rows, sm, n_rows, row_seq, conv, heads_out, out);
}
