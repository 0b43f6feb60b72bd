// Gated delta rule: a linear-attention recurrence whose state is one [dim, vdim] f32 matrix per head and
// sequence.  Per token S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q.  Both products against S are
// taken on the state before the write: S_new^T q = g S^T q + (k . q) u, so a token costs one pass over the
// state and one reduction instead of two.  Everything here is f32.
//
//   delta_step_kernel     decoding: convolution, norms, recurrence, output norm and gate of one token
//   delta_conv_kernel     prompts: convolution + silu, unit norms, decay and step size of every row
//   delta_scan_kernel     prompts: the recurrence (state columns are independent: a block owns 16 of them)
//   delta_out_kernel      prompts: output norm and gate
//
// The convolution's inputs are kept in a ring of `taps` rows per slot (position p in row p % taps): a token
// reads the other rows and replaces its own, so heads that share a query/key head do not race.
#include <algorithm>

#include "device_utils.cuh"
#include "hybrid.h"

namespace {

__device__ __forceinline__ float silu_f(float v) { return v / (1.0f + expf(-v)); }
__device__ __forceinline__ float softplus_f(float v) { return v > 20.0f ? v : log1pf(expf(v)); }
__device__ __forceinline__ float sigmoid_f(float v) { return 1.0f / (1.0f + expf(-v)); }
__device__ __forceinline__ float decay_f(float a_exp, float a, float dt_bias) { return expf(-a_exp * softplus_f(a + dt_bias)); }

// ---- decoding ----------------------------------------------------------------------------------------
// Block = (row, head), eight warps.  Warp w holds state rows w, w + 8, ...; lane l columns 4l .. 4l+3 of a
// 128-column chunk (one chunk for vdim <= 128).
template <int RPW, typename T>
__global__ void __launch_bounds__(256)
delta_step_kernel(DeltaDims d, const float *__restrict__ proj, int ldp, DeltaWeights w, float *__restrict__ conv_state,
                  float *__restrict__ state, RowMap rows, T *__restrict__ out) {
    extern __shared__ float sh[]; // q [dim_p], k [dim_p], v [vdim_p], o [vdim_p], reduction [8][2][128], scalars [8]
    const int h = blockIdx.x, row = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    float *sq = sh, *sk = sq + d.dim_p, *sv = sk + d.dim_p, *so = sv + d.vdim_p, *red = so + d.vdim_p, *sc = red + 2048;
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
    const int cw = d.conv_w();
    float *cring = conv_state + (size_t)slot * d.taps * cw;
    for (int t = tid; t < 2 * d.dim_p + d.vdim_p; t += 256) {
        const int which = t < d.dim_p ? 0 : t < 2 * d.dim_p ? 1 : 2;
        const int ch = which == 0 ? d.q_at() + kh * d.dim_p + t
                                  : which == 1 ? d.k_at() + kh * d.dim_p + (t - d.dim_p) : d.v_at() + h * d.vdim_p + (t - 2 * d.dim_p);
        const float x = p[ch];
        const float *cwt = w.conv + (size_t)ch * d.taps;
        float a = x * cwt[d.taps - 1];
        for (int j = 1; j < d.taps; ++j)
            if (pos - j >= 0) a = fmaf(cring[(size_t)((pos - j) % d.taps) * cw + ch], cwt[d.taps - 1 - j], a);
        if (which == 2 || h % group == 0) cring[(size_t)(pos % d.taps) * cw + ch] = x;
        sh[t] = silu_f(a); // q, k and v lie behind one another
    }
    __syncthreads();
    if (warp < 2) { // unit norms; q also times dim^(-1/2)
        float *x = warp ? sk : sq;
        float s = 0.0f;
        for (int j = lane; j < d.dim_p; j += 32) s = fmaf(x[j], x[j], s);
        s = warp_sum(s);
        float f = 1.0f / sqrtf(s + 1e-6f);
        if (warp == 0) f *= 1.0f / sqrtf((float)d.dim);
        for (int j = lane; j < d.dim_p; j += 32) x[j] *= f;
    } else if (tid == 64) {
        sc[0] = sigmoid_f(p[d.b_at() + h]);
        sc[1] = decay_f(w.a_exp[h], p[d.a_at() + h], w.dt_bias[h]);
    }
    __syncthreads();
    float kq = 0.0f;
    for (int j = lane; j < d.dim_p; j += 32) kq = fmaf(sk[j], sq[j], kq);
    kq = warp_sum(kq);
    const float beta = sc[0], g = sc[1];
    for (int c0 = 0; c0 < d.vdim_p; c0 += 128) {
        if (c0) load_chunk(c0);
        float4 ak = make_float4(0.f, 0.f, 0.f, 0.f), aq = ak;
#pragma unroll
        for (int r = 0; r < RPW; ++r) {
            const int i = warp + 8 * r;
            if (i < d.dim_p) {
                const float k = sk[i], q = sq[i];
                ak.x = fmaf(st[r].x, k, ak.x); ak.y = fmaf(st[r].y, k, ak.y); ak.z = fmaf(st[r].z, k, ak.z); ak.w = fmaf(st[r].w, k, ak.w);
                aq.x = fmaf(st[r].x, q, aq.x); aq.y = fmaf(st[r].y, q, aq.y); aq.z = fmaf(st[r].z, q, aq.z); aq.w = fmaf(st[r].w, q, aq.w);
            }
        }
        *reinterpret_cast<float4 *>(red + (warp * 2) * 128 + lane * 4) = ak;
        *reinterpret_cast<float4 *>(red + (warp * 2 + 1) * 128 + lane * 4) = aq;
        __syncthreads();
        float4 tk = make_float4(0.f, 0.f, 0.f, 0.f), tq = tk;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            tk = f4_add(tk, *reinterpret_cast<const float4 *>(red + (i * 2) * 128 + lane * 4));
            tq = f4_add(tq, *reinterpret_cast<const float4 *>(red + (i * 2 + 1) * 128 + lane * 4));
        }
        const int c = c0 + lane * 4;
        if (c < d.vdim_p) {
            const float4 v = *reinterpret_cast<const float4 *>(sv + c);
            const float4 u = make_float4(beta * (v.x - g * tk.x), beta * (v.y - g * tk.y), beta * (v.z - g * tk.z), beta * (v.w - g * tk.w));
            if (warp == 0)
                *reinterpret_cast<float4 *>(so + c) =
                    make_float4(fmaf(kq, u.x, g * tq.x), fmaf(kq, u.y, g * tq.y), fmaf(kq, u.z, g * tq.z), fmaf(kq, u.w, g * tq.w));
#pragma unroll
            for (int r = 0; r < RPW; ++r) {
                const int i = warp + 8 * r;
                if (i < d.dim_p) {
                    const float k = sk[i];
                    *reinterpret_cast<float4 *>(S + (size_t)i * d.vdim_p + c) =
                        make_float4(fmaf(k, u.x, g * st[r].x), fmaf(k, u.y, g * st[r].y), fmaf(k, u.z, g * st[r].z), fmaf(k, u.w, g * st[r].w));
                }
            }
        }
        __syncthreads();
    }
    float s = 0.0f; // every warp takes the sum for itself
    for (int j = lane; j < d.vdim; j += 32) s = fmaf(so[j], so[j], s);
    s = warp_sum(s);
    const float rn = 1.0f / sqrtf(s / (float)d.vdim + d.eps);
    for (int j = tid; j < d.vdim; j += 256)
        store_from_float(out + ((size_t)row * d.heads + h) * d.vdim_p + j, so[j] * rn * w.norm[j] * silu_f(p[d.g_at() + h * d.vdim_p + j]));
}

// ---- prompts -----------------------------------------------------------------------------------------
// Block = row; a warp takes one head of q, k or v at a time.
__global__ void __launch_bounds__(256)
delta_conv_kernel(DeltaDims d, const float *__restrict__ proj, int ldp, DeltaWeights w, const float *__restrict__ conv_state, RowMap rows,
                  SeqMap sm, const int *__restrict__ row_seq, float *__restrict__ conv) {
    pdl_trigger();
    pdl_wait();
    const int row = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int pos = row_pos(rows, row), slot = row_slot(rows, row), i = row - sm.row0[row_seq[row]], cw = d.conv_w();
    const float *cring = conv_state + (size_t)slot * d.taps * cw;
    float *o = conv + (size_t)row * (cw + 2 * d.heads);
    const int units = 2 * d.kv_heads + d.heads;
    for (int u = warp; u < units; u += 8) {
        const bool isv = u >= 2 * d.kv_heads;
        const int at = isv ? d.v_at() + (u - 2 * d.kv_heads) * d.vdim_p : u * d.dim_p, n = isv ? d.vdim_p : d.dim_p;
        float s = 0.0f;
        for (int j = lane; j < n; j += 32) {
            const int ch = at + j;
            const float *cwt = w.conv + (size_t)ch * d.taps;
            float a = proj[(size_t)row * ldp + ch] * cwt[d.taps - 1];
            for (int t = 1; t < d.taps; ++t) {
                if (pos - t < 0) break;
                const float x = i - t >= 0 ? proj[(size_t)(row - t) * ldp + ch] : cring[(size_t)((pos - t) % d.taps) * cw + ch];
                a = fmaf(x, cwt[d.taps - 1 - t], a);
            }
            a = silu_f(a);
            o[ch] = a;
            s = fmaf(a, a, s);
        }
        if (!isv) {
            s = warp_sum(s);
            float f = 1.0f / sqrtf(s + 1e-6f);
            if (u < d.kv_heads) f *= 1.0f / sqrtf((float)d.dim);
            for (int j = lane; j < n; j += 32) o[at + j] *= f; // the lane's own values
        }
    }
    const float *p = proj + (size_t)row * ldp;
    for (int h = threadIdx.x; h < d.heads; h += 256) {
        o[cw + h] = decay_f(w.a_exp[h], p[d.a_at() + h], w.dt_bias[h]);
        o[cw + d.heads + h] = sigmoid_f(p[d.b_at() + h]);
    }
}

// Block = (16 state columns, head, sequence), four warps of four columns; the eight lanes of a column hold its
// dim entries 4 l + 32 m .. + 3.  Tokens come through shared memory CH at a time.  Also leaves the
// convolution's last inputs in the cache (blocks of column group 0).
template <int DM>
__global__ void __launch_bounds__(128)
delta_scan_kernel(DeltaDims d, const float *__restrict__ proj, int ldp, const float *__restrict__ conv, float *__restrict__ conv_state,
                  float *__restrict__ state, SeqMap sm, float *__restrict__ heads_out) {
    constexpr int CH = DM <= 4 ? 32 : 16, DP = DM * 32;
    __shared__ __align__(16) float sk[CH][DP], sq[CH][DP];
    __shared__ float sv[CH][16], sg[CH], sb[CH], skq[CH];
    pdl_trigger();
    const int cg = blockIdx.x, h = blockIdx.y, sidx = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int cl = warp * 4 + (lane >> 3), part = lane & 7, col = cg * 16 + cl;
    pdl_wait();
    const int n = sm.n[sidx], past = sm.past[sidx], slot = sm.slot[sidx], row0 = sm.row0[sidx];
    const int group = d.heads / d.kv_heads, kh = h / group, cw = d.conv_w(), ldc = cw + 2 * d.heads;
    float *S = state + ((size_t)slot * d.heads + h) * d.dim_p * d.vdim_p + col;
    float s[DM * 4];
#pragma unroll
    for (int m = 0; m < DM; ++m)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = 32 * m + 4 * part + e;
            s[4 * m + e] = i < d.dim_p && past > 0 ? S[(size_t)i * d.vdim_p] : 0.0f;
        }
    for (int t0 = 0; t0 < n; t0 += CH) {
        const int nt = min(CH, n - t0);
        __syncthreads();
        for (int i = tid; i < nt * DP; i += 128) {
            const int t = i / DP, j = i - t * DP;
            const float *c = conv + (size_t)(row0 + t0 + t) * ldc;
            sq[t][j] = j < d.dim_p ? c[d.q_at() + kh * d.dim_p + j] : 0.0f;
            sk[t][j] = j < d.dim_p ? c[d.k_at() + kh * d.dim_p + j] : 0.0f;
        }
        for (int i = tid; i < nt * 16; i += 128)
            sv[i >> 4][i & 15] = conv[(size_t)(row0 + t0 + (i >> 4)) * ldc + d.v_at() + h * d.vdim_p + cg * 16 + (i & 15)];
        if (tid < nt) {
            sg[tid] = conv[(size_t)(row0 + t0 + tid) * ldc + cw + h];
            sb[tid] = conv[(size_t)(row0 + t0 + tid) * ldc + cw + d.heads + h];
        }
        __syncthreads();
        for (int t = warp; t < nt; t += 4) {
            float a = 0.0f;
            for (int j = lane; j < DP; j += 32) a = fmaf(sk[t][j], sq[t][j], a);
            a = warp_sum(a);
            if (lane == 0) skq[t] = a;
        }
        __syncthreads();
        for (int t = 0; t < nt; ++t) {
            float4 k[DM];
            float ak = 0.0f, aq = 0.0f;
#pragma unroll
            for (int m = 0; m < DM; ++m) {
                k[m] = *reinterpret_cast<const float4 *>(&sk[t][32 * m + 4 * part]);
                const float4 q = *reinterpret_cast<const float4 *>(&sq[t][32 * m + 4 * part]);
                ak = fmaf(s[4 * m], k[m].x, ak); ak = fmaf(s[4 * m + 1], k[m].y, ak);
                ak = fmaf(s[4 * m + 2], k[m].z, ak); ak = fmaf(s[4 * m + 3], k[m].w, ak);
                aq = fmaf(s[4 * m], q.x, aq); aq = fmaf(s[4 * m + 1], q.y, aq);
                aq = fmaf(s[4 * m + 2], q.z, aq); aq = fmaf(s[4 * m + 3], q.w, aq);
            }
#pragma unroll
            for (int o = 1; o < 8; o <<= 1) {
                ak += __shfl_xor_sync(0xffffffffu, ak, o);
                aq += __shfl_xor_sync(0xffffffffu, aq, o);
            }
            const float g = sg[t], u = sb[t] * (sv[t][cl] - g * ak);
#pragma unroll
            for (int m = 0; m < DM; ++m) {
                s[4 * m] = fmaf(k[m].x, u, g * s[4 * m]);
                s[4 * m + 1] = fmaf(k[m].y, u, g * s[4 * m + 1]);
                s[4 * m + 2] = fmaf(k[m].z, u, g * s[4 * m + 2]);
                s[4 * m + 3] = fmaf(k[m].w, u, g * s[4 * m + 3]);
            }
            if (part == 0) heads_out[((size_t)(row0 + t0 + t) * d.heads + h) * d.vdim_p + col] = fmaf(skq[t], u, g * aq);
        }
    }
#pragma unroll
    for (int m = 0; m < DM; ++m)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = 32 * m + 4 * part + e;
            if (i < d.dim_p) S[(size_t)i * d.vdim_p] = s[4 * m + e];
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
template <typename T>
__global__ void __launch_bounds__(256)
delta_out_kernel(DeltaDims d, const float *__restrict__ proj, int ldp, const float *__restrict__ norm, const float *__restrict__ heads_out,
                 int n_rows, T *__restrict__ out) {
    pdl_trigger();
    pdl_wait();
    const int unit = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (unit >= n_rows * d.heads) return;
    const int row = unit / d.heads, h = unit - row * d.heads;
    const float *o = heads_out + (size_t)unit * d.vdim_p;
    float s = 0.0f;
    for (int j = lane; j < d.vdim; j += 32) s = fmaf(o[j], o[j], s);
    s = warp_sum(s);
    const float rn = 1.0f / sqrtf(s / (float)d.vdim + d.eps);
    const float *g = proj + (size_t)row * ldp + d.g_at() + h * d.vdim_p;
    for (int j = lane; j < d.vdim; j += 32) store_from_float(out + (size_t)unit * d.vdim_p + j, o[j] * rn * norm[j] * silu_f(g[j]));
}

}  // namespace

int launch_delta_step(b200nn_ctx *ctx, const DeltaDims &d, bool b16, const float *proj, int ldp, const DeltaWeights &w, float *conv_state,
                      float *state, const RowMap &rows, int n_rows, void *out) {
    if (n_rows > 65535) return set_error(ctx, B200NN_ERR_SHAPE, "delta rule: more than 65535 rows");
    const dim3 grid(d.heads, n_rows);
    const size_t smem = (2 * d.dim_p + 2 * d.vdim_p + 2048 + 8) * sizeof(float);
#define DSTEP(R)                                                                                                             \
    do {                                                                                                                     \
        PREFER_SMEM_ONCE((delta_step_kernel<R, __nv_bfloat16>));                                                             \
        PREFER_SMEM_ONCE((delta_step_kernel<R, float>));                                                                     \
        if (b16)                                                                                                             \
            launch_pdl(ctx, delta_step_kernel<R, __nv_bfloat16>, grid, dim3(256), smem, d, proj, ldp, w, conv_state, state,  \
                       rows, (__nv_bfloat16 *)out);                                                                          \
        else                                                                                                                 \
            launch_pdl(ctx, delta_step_kernel<R, float>, grid, dim3(256), smem, d, proj, ldp, w, conv_state, state, rows,    \
                       (float *)out);                                                                                        \
    } while (0)
    if (d.dim_p <= 64) DSTEP(8);
    else if (d.dim_p <= 128) DSTEP(16);
    else if (d.dim_p <= 256) DSTEP(32);
    else return set_error(ctx, B200NN_ERR_UNSUPPORTED, "delta rule: dim > 256");
#undef DSTEP
    CK_LAUNCH(ctx, "delta_step_kernel");
    return B200NN_OK;
}

int launch_delta_prompt(b200nn_ctx *ctx, const DeltaDims &d, bool b16, const float *proj, int ldp, const DeltaWeights &w,
                        float *conv_state, float *state, const RowMap &rows, const SeqMap &sm, int n_rows, const int *row_seq, float *conv,
                        float *heads_out, void *out) {
    PREFER_SMEM_ONCE(delta_conv_kernel);
    launch_pdl(ctx, delta_conv_kernel, dim3(n_rows), dim3(256), 0, d, proj, ldp, w, conv_state, rows, sm, row_seq, conv);
    CK_LAUNCH(ctx, "delta_conv_kernel");
    const dim3 grid(d.vdim_p / 16, d.heads, sm.n_seq);
#define DSCAN(M)                                                                                                              \
    do {                                                                                                                      \
        PREFER_SMEM_ONCE(delta_scan_kernel<M>);                                                                               \
        launch_pdl(ctx, delta_scan_kernel<M>, grid, dim3(128), 0, d, proj, ldp, conv, conv_state, state, sm, heads_out);      \
    } while (0)
    const int dm = (d.dim_p + 31) / 32;
    if (dm <= 1) DSCAN(1);
    else if (dm <= 2) DSCAN(2);
    else if (dm <= 3) DSCAN(3);
    else if (dm <= 4) DSCAN(4);
    else if (dm <= 6) DSCAN(6);
    else if (dm <= 8) DSCAN(8);
    else return set_error(ctx, B200NN_ERR_UNSUPPORTED, "delta rule: dim > 256");
#undef DSCAN
    CK_LAUNCH(ctx, "delta_scan_kernel");
    const int units = n_rows * d.heads;
    if (b16) {
        PREFER_SMEM_ONCE(delta_out_kernel<__nv_bfloat16>);
        launch_pdl(ctx, delta_out_kernel<__nv_bfloat16>, dim3((units + 7) / 8), dim3(256), 0, d, proj, ldp, w.norm, heads_out, n_rows,
                   (__nv_bfloat16 *)out);
    } else {
        PREFER_SMEM_ONCE(delta_out_kernel<float>);
        launch_pdl(ctx, delta_out_kernel<float>, dim3((units + 7) / 8), dim3(256), 0, d, proj, ldp, w.norm, heads_out, n_rows, (float *)out);
    }
    CK_LAUNCH(ctx, "delta_out_kernel");
    return B200NN_OK;
}
