// Latent attention: what happens between its matrix products.
//
// A token's key and value are products of one small latent per token, so the cache holds the normalised latent
// and one rotated key part shared by all heads.  Prompt passes expand the window's latents to keys and values
// once (a GEMM) and attend over those; decoding stays in the latent space: the query is taken through the key
// up-projection once, every head then scores and sums the same cached rows, and the value up-projection
// follows the softmax.
//
// The cache is a ring of rows per slot (position p in row p % ring).  A windowed layer's ring holds the window
// plus the longest prompt portion, so a portion's first query still finds its oldest key after the portion's
// own rows have been written.
#include <algorithm>

#include "device_utils.cuh"
#include "hybrid.h"

namespace {

template <typename T>
__global__ void __launch_bounds__(128)
latent_prep_kernel(LatentDims d, const float *__restrict__ proj, int ldp, const float *__restrict__ q_norm,
                   const float *__restrict__ kv_norm, const float2 *__restrict__ rope, RowMap rows, T *__restrict__ cq,
                   T *__restrict__ cache, int ring, float *__restrict__ gate) {
    __shared__ float red[2];
    pdl_trigger();
    pdl_wait();
    const int r = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const float *p = proj + (size_t)r * ldp, *pc = p + d.q_rank, *pr = pc + d.rank, *pg = pr + d.rot;
    if (warp < 2) { // one warp per norm
        const float *src = warp ? pc : p;
        const int n = warp ? d.rank : d.q_rank;
        float s = 0.0f;
        for (int j = lane; j < n; j += 32) s = fmaf(src[j], src[j], s);
        s = warp_sum(s);
        if (lane == 0) red[warp] = 1.0f / sqrtf(s / (float)n + d.eps);
    }
    __syncthreads();
    const float rq = red[0], rc = red[1];
    T *q = cq + (size_t)r * d.q_rank_p;
    for (int j = tid; j < d.q_rank; j += 128) store_from_float(q + j, p[j] * rq * q_norm[j]);
    const int pos = row_pos(rows, r);
    T *c = cache + ((size_t)row_slot(rows, r) * ring + pos % ring) * (d.rank_p + d.rot_p);
    for (int j = tid; j < d.rank_p; j += 128) store_from_float(c + j, j < d.rank ? pc[j] * rc * kv_norm[j] : 0.0f);
    const int half = d.rot >> 1;
    for (int i = tid; i < d.rot_p >> 1; i += 128) {
        float u = 0.0f, v = 0.0f;
        if (i < half) {
            const float2 cs = rope[(size_t)pos * half + i];
            const float a = pr[i], b = pr[i + half];
            u = a * cs.x - b * cs.y;
            v = b * cs.x + a * cs.y;
        }
        store_from_float(c + d.rank_p + 2 * i, u);
        store_from_float(c + d.rank_p + 2 * i + 1, v);
    }
    for (int h = tid; h < d.heads; h += 128) gate[(size_t)r * d.heads + h] = 1.0f / (1.0f + expf(-pg[h]));
}

__global__ void rope_heads_kernel(float *__restrict__ q, int n_rows, int heads, int head_w, int at, int pairs,
                                  const float2 *__restrict__ tab, RowMap rows) {
    pdl_trigger();
    pdl_wait();
    const int total = n_rows * heads * pairs;
    for (int t = blockIdx.x * blockDim.x + threadIdx.x; t < total; t += gridDim.x * blockDim.x) {
        const int i = t % pairs, h = (t / pairs) % heads, r = t / (pairs * heads);
        float *x = q + ((size_t)r * heads + h) * head_w + at + 2 * i;
        const float2 cs = tab[(size_t)row_pos(rows, r) * pairs + i];
        const float u = x[0], v = x[1];
        x[0] = u * cs.x - v * cs.y;
        x[1] = v * cs.x + u * cs.y;
    }
}

// 16-byte pieces: rows are multiples of 32 bytes.
__global__ void latent_gather_kernel(const uint4 *__restrict__ cache, int ring, int pieces, SeqMap sm, uint4 *__restrict__ lin) {
    pdl_trigger();
    pdl_wait();
    const int s = blockIdx.y, klen = sm.klen[s];
    const size_t slot = (size_t)sm.slot[s] * ring;
    for (int t = blockIdx.x * blockDim.x + threadIdx.x; t < klen * pieces; t += gridDim.x * blockDim.x) {
        const int j = t / pieces, c = t - j * pieces;
        lin[(size_t)(sm.krow0[s] + j) * pieces + c] = cache[(slot + (sm.kpos0[s] + j) % ring) * pieces + c];
    }
}

// One block per (head, prompt row): 128 keys at a time with a running softmax.
template <typename T>
__global__ void __launch_bounds__(128)
latent_prefill_simple_kernel(LatentDims d, const T *__restrict__ q, const T *__restrict__ kvx, const T *__restrict__ lin, SeqMap sm,
                             const float *__restrict__ gate, T *__restrict__ out) {
    extern __shared__ float sh[]; // query [head_w], weights [128], red [8]
    pdl_trigger();
    pdl_wait();
    const int h = blockIdx.x, s = blockIdx.z, i = blockIdx.y, tid = threadIdx.x;
    if (i >= sm.n[s]) return;
    const int hw = d.dim_p + d.rot_p, ld = d.rank_p + d.rot_p, kvw = d.heads * (d.dim_p + d.vdim_p);
    float *sq = sh, *sp = sh + hw, *red = sp + 128;
    const int row = sm.row0[s] + i, pos = sm.past[s] + i;
    const T *qr = q + ((size_t)row * d.heads + h) * hw;
    for (int j = tid; j < hw; j += 128) sq[j] = load_as_float<T>(qr, j);
    __syncthreads();
    const int first = d.window ? max(0, pos - d.window + 1) : 0;
    float m = -INFINITY, l = 0.0f, acc[4] = {0.f, 0.f, 0.f, 0.f}; // vdim_p <= 512
    for (int k0 = first; k0 <= pos; k0 += 128) {
        const int n = min(128, pos - k0 + 1);
        const size_t kr = (size_t)sm.krow0[s] + (k0 - sm.kpos0[s]);
        float sc = -INFINITY;
        if (tid < n) {
            const T *kn = kvx + (kr + tid) * kvw + h * d.dim_p;
            const T *kro = lin + (kr + tid) * ld + d.rank_p;
            float a = 0.0f;
            for (int j = 0; j < d.dim_p; ++j) a = fmaf(sq[j], load_as_float<T>(kn, j), a);
            for (int j = 0; j < d.rot; ++j) a = fmaf(sq[d.dim_p + j], load_as_float<T>(kro, j), a);
            sc = a * d.scale;
        }
        float mx = warp_max(sc);
        if ((tid & 31) == 0) red[tid >> 5] = mx;
        __syncthreads();
        mx = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
        const float m_new = fmaxf(m, mx), corr = expf(m - m_new);
        const float p = tid < n ? expf(sc - m_new) : 0.0f;
        sp[tid] = p;
        const float ps = warp_sum(p);
        if ((tid & 31) == 0) red[4 + (tid >> 5)] = ps;
        __syncthreads();
        l = l * corr + ((red[4] + red[5]) + (red[6] + red[7]));
        m = m_new;
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const int e = tid + 128 * c;
            if (e < d.vdim_p) {
                const T *v = kvx + kr * kvw + d.heads * d.dim_p + h * d.vdim_p + e;
                float a = acc[c] * corr;
                for (int j = 0; j < n; ++j) a = fmaf(sp[j], load_as_float<T>(v, (size_t)j * kvw), a);
                acc[c] = a;
            }
        }
        __syncthreads();
    }
    const float f = gate[(size_t)row * d.heads + h] / l;
#pragma unroll
    for (int c = 0; c < 4; ++c) {
        const int e = tid + 128 * c;
        if (e < d.vdim_p) store_from_float(out + ((size_t)row * d.heads + h) * d.vdim_p + e, acc[c] * f);
    }
}

// One block per (head, row): as above over cached latents.
template <typename T>
__global__ void __launch_bounds__(128)
latent_decode_simple_kernel(LatentDims d, const T *__restrict__ q, const T *__restrict__ qlat, const T *__restrict__ cache, int ring,
                            RowMap rows, T *__restrict__ out) {
    extern __shared__ float sh[]; // query [rank_p + rot_p], weights [128], red [8]
    pdl_trigger();
    pdl_wait();
    const int h = blockIdx.x, row = blockIdx.y, tid = threadIdx.x;
    const int hw = d.dim_p + d.rot_p, ld = d.rank_p + d.rot_p;
    float *sq = sh, *sp = sh + ld, *red = sp + 128;
    const T *ql = qlat + ((size_t)row * d.heads + h) * d.rank_p, *qr = q + ((size_t)row * d.heads + h) * hw + d.dim_p;
    for (int j = tid; j < d.rank_p; j += 128) sq[j] = load_as_float<T>(ql, j);
    for (int j = tid; j < d.rot_p; j += 128) sq[d.rank_p + j] = load_as_float<T>(qr, j);
    __syncthreads();
    const int pos = row_pos(rows, row), first = d.window ? max(0, pos - d.window + 1) : 0;
    const T *base = cache + (size_t)row_slot(rows, row) * ring * ld;
    float m = -INFINITY, l = 0.0f, acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f}; // rank_p <= 1024
    for (int k0 = first; k0 <= pos; k0 += 128) {
        const int n = min(128, pos - k0 + 1);
        float sc = -INFINITY;
        if (tid < n) {
            const T *k = base + (size_t)((k0 + tid) % ring) * ld;
            float a = 0.0f;
            for (int j = 0; j < ld; ++j) a = fmaf(sq[j], load_as_float<T>(k, j), a);
            sc = a * d.scale;
        }
        float mx = warp_max(sc);
        if ((tid & 31) == 0) red[tid >> 5] = mx;
        __syncthreads();
        mx = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
        const float m_new = fmaxf(m, mx), corr = expf(m - m_new);
        const float p = tid < n ? expf(sc - m_new) : 0.0f;
        sp[tid] = p;
        const float ps = warp_sum(p);
        if ((tid & 31) == 0) red[4 + (tid >> 5)] = ps;
        __syncthreads();
        l = l * corr + ((red[4] + red[5]) + (red[6] + red[7]));
        m = m_new;
#pragma unroll
        for (int c = 0; c < 8; ++c) {
            const int e = tid + 128 * c;
            if (e < d.rank_p) {
                float a = acc[c] * corr;
                int kr = k0 % ring;
                for (int j = 0; j < n; ++j) {
                    a = fmaf(sp[j], load_as_float<T>(base + (size_t)kr * ld, e), a);
                    if (++kr == ring) kr = 0;
                }
                acc[c] = a;
            }
        }
        __syncthreads();
    }
    const float f = 1.0f / l;
#pragma unroll
    for (int c = 0; c < 8; ++c) {
        const int e = tid + 128 * c;
        if (e < d.rank_p) store_from_float(out + ((size_t)row * d.heads + h) * d.rank_p + e, acc[c] * f);
    }
}

}  // namespace

int launch_latent_prep(b200nn_ctx *ctx, const LatentDims &d, bool b16, const float *proj, int ldp, const float *q_norm,
                       const float *kv_norm, const float2 *rope, const RowMap &rows, int n_rows, void *cq, void *cache, int ring,
                       float *gate) {
    if (b16) {
        PREFER_SMEM_ONCE(latent_prep_kernel<__nv_bfloat16>);
        launch_pdl(ctx, latent_prep_kernel<__nv_bfloat16>, dim3(n_rows), dim3(128), 0, d, proj, ldp, q_norm, kv_norm, rope, rows,
                   (__nv_bfloat16 *)cq, (__nv_bfloat16 *)cache, ring, gate);
    } else {
        PREFER_SMEM_ONCE(latent_prep_kernel<float>);
        launch_pdl(ctx, latent_prep_kernel<float>, dim3(n_rows), dim3(128), 0, d, proj, ldp, q_norm, kv_norm, rope, rows, (float *)cq,
                   (float *)cache, ring, gate);
    }
    CK_LAUNCH(ctx, "latent_prep_kernel");
    return B200NN_OK;
}

int launch_rope_heads(b200nn_ctx *ctx, float *q, int n_rows, int heads, int head_w, int at, int pairs, const float2 *tab,
                      const RowMap &rows) {
    const long long total = (long long)n_rows * heads * pairs;
    if (total <= 0) return B200NN_OK;
    PREFER_SMEM_ONCE(rope_heads_kernel);
    launch_pdl(ctx, rope_heads_kernel, dim3((unsigned)std::min<long long>((total + 255) / 256, 4096)), dim3(256), 0, q, n_rows, heads,
               head_w, at, pairs, tab, rows);
    CK_LAUNCH(ctx, "rope_heads_kernel");
    return B200NN_OK;
}

int launch_latent_gather(b200nn_ctx *ctx, const LatentDims &d, bool b16, const void *cache, int ring, const SeqMap &sm, void *lin) {
    const int pieces = d.ld() * (b16 ? 2 : 4) / 16;
    const int blocks = std::max(1, std::min(256, (sm.max_k * pieces + 255) / 256));
    PREFER_SMEM_ONCE(latent_gather_kernel);
    launch_pdl(ctx, latent_gather_kernel, dim3(blocks, sm.n_seq), dim3(256), 0, (const uint4 *)cache, ring, pieces, sm, (uint4 *)lin);
    CK_LAUNCH(ctx, "latent_gather_kernel");
    return B200NN_OK;
}

int launch_latent_prefill(b200nn_ctx *ctx, const LatentDims &d, bool b16, int n_rows, const void *q, const void *kvx, const void *lin,
                          const SeqMap &sm, const float *gate, void *out) {
    if (b16 && latent_prefill_tc_supported(ctx, d))
        return launch_latent_prefill_tc(ctx, d, n_rows, (const __nv_bfloat16 *)q, (const __nv_bfloat16 *)kvx, (const __nv_bfloat16 *)lin, sm, gate,
                                        (__nv_bfloat16 *)out);
    if (d.vdim_p > 512) return set_error(ctx, B200NN_ERR_UNSUPPORTED, "latent attention: vdim > 512");
    const dim3 grid(d.heads, sm.max_n, sm.n_seq);
    if (sm.max_n > 65535 || sm.n_seq > 65535) return set_error(ctx, B200NN_ERR_SHAPE, "latent attention: more than 65535 rows or sequences");
    const size_t smem = (d.head_w() + 136) * sizeof(float);
    if (b16) {
        PREFER_SMEM_ONCE(latent_prefill_simple_kernel<__nv_bfloat16>);
        launch_pdl(ctx, latent_prefill_simple_kernel<__nv_bfloat16>, grid, dim3(128), smem, d, (const __nv_bfloat16 *)q,
                   (const __nv_bfloat16 *)kvx, (const __nv_bfloat16 *)lin, sm, gate, (__nv_bfloat16 *)out);
    } else {
        PREFER_SMEM_ONCE(latent_prefill_simple_kernel<float>);
        launch_pdl(ctx, latent_prefill_simple_kernel<float>, grid, dim3(128), smem, d, (const float *)q, (const float *)kvx,
                   (const float *)lin, sm, gate, (float *)out);
    }
    CK_LAUNCH(ctx, "latent_prefill_simple_kernel");
    return B200NN_OK;
}

size_t latent_decode_part_floats(const b200nn_ctx *ctx, const LatentDims &d, bool b16, int n_rows, int cap) {
    return b16 && latent_decode_tc_supported(ctx, d) ? latent_decode_tc_part_floats(ctx, d, n_rows, cap) : 0;
}

int launch_latent_decode(b200nn_ctx *ctx, const LatentDims &d, bool b16, const void *q, const void *qlat, const void *cache, int ring,
                         size_t cache_rows, const RowMap &rows, int n_rows, int cap, void *out, float *part) {
    if (b16 && latent_decode_tc_supported(ctx, d))
        return launch_latent_decode_tc(ctx, d, (const __nv_bfloat16 *)q, (const __nv_bfloat16 *)qlat, (const __nv_bfloat16 *)cache, ring, cache_rows,
                                       rows, n_rows, cap, (__nv_bfloat16 *)out, part);
    if (d.rank_p > 1024) return set_error(ctx, B200NN_ERR_UNSUPPORTED, "latent attention: kv_rank > 1024");
    if (n_rows > 65535) return set_error(ctx, B200NN_ERR_SHAPE, "latent attention: more than 65535 rows");
    const dim3 grid(d.heads, n_rows);
    const size_t smem = (d.ld() + 136) * sizeof(float);
    if (b16) {
        PREFER_SMEM_ONCE(latent_decode_simple_kernel<__nv_bfloat16>);
        launch_pdl(ctx, latent_decode_simple_kernel<__nv_bfloat16>, grid, dim3(128), smem, d, (const __nv_bfloat16 *)q,
                   (const __nv_bfloat16 *)qlat, (const __nv_bfloat16 *)cache, ring, rows, (__nv_bfloat16 *)out);
    } else {
        PREFER_SMEM_ONCE(latent_decode_simple_kernel<float>);
        launch_pdl(ctx, latent_decode_simple_kernel<float>, grid, dim3(128), smem, d, (const float *)q, (const float *)qlat,
                   (const float *)cache, ring, rows, (float *)out);
    }
    CK_LAUNCH(ctx, "latent_decode_simple_kernel");
    return B200NN_OK;
}
