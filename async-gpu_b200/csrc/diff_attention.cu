// Differential attention: two softmax maps per head over the same values, subtracted, normalised and gated (DiffDims in
// hybrid.h).  This file has the CUDA-core form, which serves f32 models and sizes beyond the tensor-core kernels
// (diff_attention_tc.cu for prompts, diff_decode_tc.cu for decoding), and the dispatch.
#include <algorithm>

#include "device_utils.cuh"
#include "hybrid.h"

namespace {

// One block per (head, row), prompts and decoding alike: 128 keys at a time, running softmaxes of both maps.
template <typename T>
__global__ void __launch_bounds__(128)
diff_simple_kernel(DiffDims d, const T *__restrict__ q, int ldq, const T *__restrict__ cache, int cap, RowMap rows, const float *__restrict__ gate, int gate_ld,
                   T *__restrict__ out) {
    extern __shared__ float sh[]; // query [2 dim_p], weights [2][128], reduction [16]
    pdl_trigger();
    pdl_wait();
    const int h = blockIdx.x, row = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int kw = d.kv_w();
    float *sq = sh, *sp = sq + 2 * d.dim_p, *red = sp + 256;
    const int pos = row_pos(rows, row);
    const float scale = d.score_scale(pos);
    for (int j = tid; j < 2 * d.dim_p; j += 128) sq[j] = load_as_float<T>(q, (size_t)row * ldq + h * 2 * d.dim_p + j);
    __syncthreads();
    const T *base = cache + ((size_t)row_slot(rows, row) * d.kv_heads + h / d.group()) * cap * kw;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f}, acc[2][4] = {}; // vdim_p <= 512
    for (int k0 = 0; k0 <= pos; k0 += 128) {
        const int n = min(128, pos - k0 + 1);
        float s[2] = {-INFINITY, -INFINITY};
        if (tid < n) {
            const T *k = base + (size_t)(k0 + tid) * kw;
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                float a = 0.0f;
                for (int j = 0; j < d.dim_p; ++j) a = fmaf(sq[x * d.dim_p + j], load_as_float<T>(k, x * d.dim_p + j), a);
                a *= scale;
                s[x] = d.cap > 0.0f ? d.cap * tanhf(a / d.cap) : a;
            }
        }
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const float mx = warp_max(s[x]);
            if (lane == 0) red[x * 4 + warp] = mx;
        }
        __syncthreads();
        float corr[2];
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const float mn = fmaxf(m[x], fmaxf(fmaxf(red[x * 4], red[x * 4 + 1]), fmaxf(red[x * 4 + 2], red[x * 4 + 3])));
            corr[x] = expf(m[x] - mn);
            m[x] = mn;
            const float p = tid < n ? expf(s[x] - mn) : 0.0f;
            sp[x * 128 + tid] = p;
            const float ps = warp_sum(p);
            if (lane == 0) red[8 + x * 4 + warp] = ps;
        }
        __syncthreads();
#pragma unroll
        for (int x = 0; x < 2; ++x) l[x] = l[x] * corr[x] + ((red[8 + x * 4] + red[9 + x * 4]) + (red[10 + x * 4] + red[11 + x * 4]));
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const int e = tid + 128 * c;
            if (e < d.vdim_p) {
                const T *v = base + (size_t)k0 * kw + 2 * d.dim_p + e;
                float a = acc[0][c] * corr[0], b = acc[1][c] * corr[1];
                for (int j = 0; j < n; ++j) {
                    const float vv = load_as_float<T>(v, (size_t)j * kw);
                    a = fmaf(sp[j], vv, a);
                    b = fmaf(sp[128 + j], vv, b);
                }
                acc[0][c] = a;
                acc[1][c] = b;
            }
        }
        __syncthreads();
    }
    float o[4], ss = 0.0f;
#pragma unroll
    for (int c = 0; c < 4; ++c) { // columns past vdim hold zeros
        o[c] = acc[0][c] / l[0] - d.lambda * (acc[1][c] / l[1]);
        ss = fmaf(o[c], o[c], ss);
    }
    ss = warp_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    ss = (red[0] + red[1]) + (red[2] + red[3]);
    const float f = (1.0f - d.diff) * sigmoid_f(gate[(size_t)row * gate_ld + h]) / sqrtf(ss / (float)d.vdim + d.eps);
#pragma unroll
    for (int c = 0; c < 4; ++c) {
        const int e = tid + 128 * c;
        if (e < d.vdim_p) store_from_float(out + ((size_t)row * d.heads + h) * d.vdim_p + e, o[c] * f);
    }
}

__global__ void __launch_bounds__(256) kv_store_f32_kernel(const float *__restrict__ proj, int ldp, int at, int kv_heads, int kv_w, int cap, RowMap rows,
                                                           float *__restrict__ cache) {
    pdl_trigger();
    pdl_wait();
    const int r = blockIdx.x, w = kv_heads * kv_w;
    for (int c = threadIdx.x; c < w; c += 256) {
        const int g = c / kv_w;
        cache[(((size_t)row_slot(rows, r) * kv_heads + g) * cap + row_pos(rows, r)) * kv_w + (c - g * kv_w)] = proj[(size_t)r * ldp + at + c];
    }
}

}  // namespace

int launch_kv_store_f32(b200nn_ctx *ctx, const float *proj, int ldp, int at, int kv_heads, int kv_w, int cap, const RowMap &rows, int n_rows,
                        float *cache) {
    PREFER_SMEM_ONCE(kv_store_f32_kernel);
    launch_pdl(ctx, kv_store_f32_kernel, dim3(n_rows), dim3(256), 0, proj, ldp, at, kv_heads, kv_w, cap, rows, cache);
    CK_LAUNCH(ctx, "kv_store_f32_kernel");
    return B200NN_OK;
}

size_t diff_part_floats(const b200nn_ctx *ctx, const DiffDims &d, bool b16, int n_rows, int cap) {
    return b16 && diff_decode_tc_supported(ctx, d) ? diff_decode_tc_part_floats(ctx, d, n_rows, cap) : 0;
}

int launch_diff_attention(b200nn_ctx *ctx, const DiffDims &d, bool b16, const void *q, int ldq, const void *cache, int cap, size_t cache_rows,
                          const RowMap &rows, const SeqMap &sm, int n_rows, const float *gate, int gate_ld, float *part, void *out) {
    if (b16 && sm.n_seq && diff_prefill_tc_supported(ctx, d))
        return launch_diff_prefill_tc(ctx, d, (const __nv_bfloat16 *)q, ldq, (const __nv_bfloat16 *)cache, cap, cache_rows, sm, n_rows, gate, gate_ld,
                                      (__nv_bfloat16 *)out);
    if (b16 && !sm.n_seq && diff_decode_tc_supported(ctx, d))
        return launch_diff_decode_tc(ctx, d, (const __nv_bfloat16 *)q, ldq, (const __nv_bfloat16 *)cache, cap, cache_rows, rows, n_rows, gate, gate_ld,
                                     part, (__nv_bfloat16 *)out);
    if (d.vdim_p > 512) return set_error(ctx, B200NN_ERR_UNSUPPORTED, "differential attention: vdim > 512");
    if (n_rows > 65535) return set_error(ctx, B200NN_ERR_SHAPE, "differential attention: more than 65535 rows");
    const dim3 grid(d.heads, n_rows);
    const size_t smem = (2 * d.dim_p + 256 + 16) * sizeof(float);
    if (b16) {
        PREFER_SMEM_ONCE(diff_simple_kernel<__nv_bfloat16>);
        launch_pdl(ctx, diff_simple_kernel<__nv_bfloat16>, grid, dim3(128), smem, d, (const __nv_bfloat16 *)q, ldq, (const __nv_bfloat16 *)cache, cap, rows,
                   gate, gate_ld, (__nv_bfloat16 *)out);
    } else {
        PREFER_SMEM_ONCE(diff_simple_kernel<float>);
        launch_pdl(ctx, diff_simple_kernel<float>, grid, dim3(128), smem, d, (const float *)q, ldq, (const float *)cache, cap, rows, gate, gate_ld,
                   (float *)out);
    }
    CK_LAUNCH(ctx, "diff_simple_kernel");
    return B200NN_OK;
}
