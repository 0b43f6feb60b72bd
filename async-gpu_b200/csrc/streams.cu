// Residual streams (hyper-connections): instead of one residual x there are n copies x_1 .. x_n per row.  A sublayer
// reads u = sum_s in[s] x_s; its output y goes back as x_t <- sum_s mix[s][t] x_s + out[t] y.
//
// One kernel per sublayer boundary does the update of the sublayer before it, the weighted sum the next sublayer
// reads and that sublayer's RMS norm, so the streams are read and written once: block = row, a thread owns columns
// of all streams.  At the ends of the model it copies the embedding into the streams, or leaves their sum.
#include "device_utils.cuh"
#include "hybrid.h"

namespace {

template <int V> struct Vec;
template <> struct Vec<4> { using type = float4; };
template <> struct Vec<1> { using type = float; };

template <int V>
__device__ __forceinline__ void load_cols(const float *p, float (&f)[V]) {
    *reinterpret_cast<typename Vec<V>::type *>(f) = *reinterpret_cast<const typename Vec<V>::type *>(p);
}
template <int V>
__device__ __forceinline__ void store_cols(float *p, const float (&f)[V]) {
    *reinterpret_cast<typename Vec<V>::type *>(p) = *reinterpret_cast<const typename Vec<V>::type *>(f);
}

// S: streams at most; V: columns per access; NV: accesses per thread; NT: threads
template <int S, int V, int NV, int NT, typename T>
__global__ void __launch_bounds__(NT)
stream_step_kernel(int n, int d, float *__restrict__ xs, const float *__restrict__ x0, const float *__restrict__ y, StreamCoef prev, StreamCoef next,
                   const float *__restrict__ norm, float eps, int ldo, T *__restrict__ out, float *__restrict__ x_sum) {
    __shared__ float red[32];
    const int row = blockIdx.x, tid = threadIdx.x;
    pdl_trigger();
    // coefficients are constant: fetched before the wait
    float mix[S][S], co[S], ci[S];
#pragma unroll
    for (int t = 0; t < S; ++t) {
        co[t] = y && t < n ? prev.out[t] : 0.0f;
        ci[t] = t < n ? (x_sum ? 1.0f : next.in[t]) : 0.0f;
#pragma unroll
        for (int s = 0; s < S; ++s) mix[s][t] = y && s < n && t < n ? prev.mix[s * n + t] : 0.0f;
    }
    pdl_wait();
    float *xr = xs + (size_t)row * n * d;
    float u[NV][V], sum = 0.0f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = (tid + i * NT) * V;
#pragma unroll
        for (int e = 0; e < V; ++e) u[i][e] = 0.0f;
        if (c >= d) continue;
        float o[S][V];
        if (y) {
            float x[S][V], yy[V];
            load_cols<V>(y + (size_t)row * d + c, yy);
#pragma unroll
            for (int s = 0; s < S; ++s)
                if (s < n) load_cols<V>(xr + (size_t)s * d + c, x[s]);
                else
#pragma unroll
                    for (int e = 0; e < V; ++e) x[s][e] = 0.0f;
#pragma unroll
            for (int t = 0; t < S; ++t)
#pragma unroll
                for (int e = 0; e < V; ++e) {
                    float a = co[t] * yy[e];
#pragma unroll
                    for (int s = 0; s < S; ++s) a = fmaf(mix[s][t], x[s][e], a);
                    o[t][e] = a;
                }
        } else {
            float x[V];
            load_cols<V>(x0 + (size_t)row * d + c, x);
#pragma unroll
            for (int t = 0; t < S; ++t)
#pragma unroll
                for (int e = 0; e < V; ++e) o[t][e] = x[e];
        }
#pragma unroll
        for (int t = 0; t < S; ++t)
            if (t < n) {
                if (!x_sum) store_cols<V>(xr + (size_t)t * d + c, o[t]);
#pragma unroll
                for (int e = 0; e < V; ++e) u[i][e] = fmaf(ci[t], o[t][e], u[i][e]);
            }
        if (x_sum) store_cols<V>(x_sum + (size_t)row * d + c, u[i]);
#pragma unroll
        for (int e = 0; e < V; ++e) sum = fmaf(u[i][e], u[i][e], sum);
    }
    if (x_sum) return;
    const float r = 1.0f / sqrtf(block_sum(sum, red) / (float)d + eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = (tid + i * NT) * V;
        if (c >= d) continue;
        float g[V];
        load_cols<V>(norm + c, g);
#pragma unroll
        for (int e = 0; e < V; ++e) g[e] *= u[i][e] * r;
        T *dst = out + (size_t)row * ldo + c;
        if constexpr (V == 4 && sizeof(T) == 2) {
            *reinterpret_cast<uint2 *>(dst) = make_uint2(pack_bf16x2(g[0], g[1]), pack_bf16x2(g[2], g[3]));
        } else {
#pragma unroll
            for (int e = 0; e < V; ++e) store_from_float(dst + e, g[e]);
        }
    }
}

template <int S, int V, int NV, int NT>
void launch_s(b200nn_ctx *ctx, const StreamStep &a, bool b16) {
    if (b16) {
        PREFER_SMEM_ONCE((stream_step_kernel<S, V, NV, NT, __nv_bfloat16>));
        launch_pdl(ctx, stream_step_kernel<S, V, NV, NT, __nv_bfloat16>, dim3(a.rows), dim3(NT), 0, a.n, a.d, a.xs, a.x0, a.y, a.prev, a.next, a.norm,
                   a.eps, a.ldo, (__nv_bfloat16 *)a.out, a.x_sum);
    } else {
        PREFER_SMEM_ONCE((stream_step_kernel<S, V, NV, NT, float>));
        launch_pdl(ctx, stream_step_kernel<S, V, NV, NT, float>, dim3(a.rows), dim3(NT), 0, a.n, a.d, a.xs, a.x0, a.y, a.prev, a.next, a.norm, a.eps,
                   a.ldo, (float *)a.out, a.x_sum);
    }
}

template <int S>
void launch_v(b200nn_ctx *ctx, const StreamStep &a, bool b16) {
    constexpr int WIDE = S <= 4 ? 1024 : 512; // threads per row of a decode step's few rows
    if (a.d % 4 || a.ldo % 4) launch_s<S, 1, 32, 256>(ctx, a, b16);
    else if (a.d <= 1024) launch_s<S, 4, 1, 256>(ctx, a, b16);
    else if (a.rows <= ctx->sm_count && a.d <= 4 * WIDE) launch_s<S, 4, 1, WIDE>(ctx, a, b16);
    else if (a.rows <= ctx->sm_count) launch_s<S, 4, 8192 / (4 * WIDE), WIDE>(ctx, a, b16);
    else if (a.d <= 2048) launch_s<S, 4, 2, 256>(ctx, a, b16);
    else if (a.d <= 4096) launch_s<S, 4, 4, 256>(ctx, a, b16);
    else launch_s<S, 4, 8, 256>(ctx, a, b16);
}

}  // namespace

int launch_stream_step(b200nn_ctx *ctx, const StreamStep &a, bool b16) {
    if (a.rows <= 0) return B200NN_OK;
    if (a.n < 1 || a.n > MAX_STREAMS) return set_error(ctx, B200NN_ERR_UNSUPPORTED, "residual streams: 1 to 8 streams");
    if (a.d > 8192) return set_error(ctx, B200NN_ERR_UNSUPPORTED, "residual streams: width > 8192");
    if (a.n == 1) launch_v<1>(ctx, a, b16);
    else if (a.n == 2) launch_v<2>(ctx, a, b16);
    else if (a.n == 3) launch_v<3>(ctx, a, b16);
    else if (a.n == 4) launch_v<4>(ctx, a, b16);
    else launch_v<8>(ctx, a, b16);
    CK_LAUNCH(ctx, "stream_step_kernel");
    return B200NN_OK;
}
