// Layer mechanisms of the hybrid decoder (hybrid.cu): gated delta rule and latent attention.
#pragma once
#include "model.h"

#define HD __host__ __device__

// The sequences of a prompt pass on the device: entry i is `n[i]` rows starting at pass row row0[i], at
// positions past[i] .. of the sequence in cache slot slot[i]; its window keys are klen[i] gathered rows from
// krow0[i] on, the first of them position kpos0[i].
struct SeqMap {
    int n_seq = 0, max_n = 0, max_k = 0, k_rows = 0;
    const int *slot = nullptr, *row0 = nullptr, *n = nullptr, *past = nullptr, *krow0 = nullptr, *klen = nullptr, *kpos0 = nullptr;
};

// ---- latent attention ----------------------------------------------------------------------------
// Column layout of its matrices (everything padded to multiples of 16 with zeros):
//   query        [row][head][dim_p unrotated | rot_p rotated, (u, v) pairs adjacent]   head_w = dim_p + rot_p
//   cache row    [rank_p latent | rot_p rotated key part]                              ld = rank_p + rot_p
//   expanded     [row][head][dim_p] keys, then [head][vdim_p] values
struct LatentDims {
    int heads, dim_p, rot, rot_p, vdim_p, rank, rank_p, q_rank, q_rank_p, window; // window 0: no limit
    float scale, eps;
    HD int head_w() const { return dim_p + rot_p; }
    HD int ld() const { return rank_p + rot_p; }
    HD int kv_w() const { return heads * (dim_p + vdim_p); }
};
// The fused down projection's rows [q_rank | rank | rot | heads] (f32, ldp apart) become the normalised query
// latent cq [row][q_rank_p], the cache rows of the tokens and the output gates sigmoid(.) [row][heads].
int launch_latent_prep(b200nn_ctx *ctx, const LatentDims &d, bool b16, const float *proj, int ldp, const float *q_norm,
                       const float *kv_norm, const float2 *rope, const RowMap &rows, int n_rows, void *cq, void *cache, int ring,
                       float *gate);
// In-place rotation of a query matrix's rotated columns (f32 models; bfloat16 ones rotate in the epilogue).
int launch_rope_heads(b200nn_ctx *ctx, float *q, int n_rows, int heads, int head_w, int at, int pairs, const float2 *tab,
                      const RowMap &rows);
// Cache rows of each sequence's window keys -> lin [k_rows][ld].
int launch_latent_gather(b200nn_ctx *ctx, const LatentDims &d, bool b16, const void *cache, int ring, const SeqMap &sm, void *lin);
// Attention of prompt rows over expanded keys and values; out [row][head][vdim_p] times the gate.
int launch_latent_prefill(b200nn_ctx *ctx, const LatentDims &d, bool b16, int n_rows, const void *q, const void *kvx, const void *lin,
                          const SeqMap &sm, const float *gate, void *out);
// Its tensor-core form (latent_attention_tc.cu): bfloat16, dim and vdim up to 128, rot_dim up to 64.
bool latent_prefill_tc_supported(const b200nn_ctx *ctx, const LatentDims &d);
int launch_latent_prefill_tc(b200nn_ctx *ctx, const LatentDims &d, int n_rows, const __nv_bfloat16 *q, const __nv_bfloat16 *kvx,
                             const __nv_bfloat16 *lin, const SeqMap &sm, const float *gate, __nv_bfloat16 *out);
// One query row per sequence against the cached latents: qlat [row][head][rank_p] (the unrotated query through
// the key up-projection), q for the rotated part; out [row][head][rank_p], the attention-weighted latents.
// cache_rows: all rows of the cache; cap bounds the positions; part: latent_decode_part_floats of scratch.
int launch_latent_decode(b200nn_ctx *ctx, const LatentDims &d, bool b16, const void *q, const void *qlat, const void *cache, int ring,
                         size_t cache_rows, const RowMap &rows, int n_rows, int cap, void *out, float *part);
size_t latent_decode_part_floats(const b200nn_ctx *ctx, const LatentDims &d, bool b16, int n_rows, int cap);
// Its tensor-core form (latent_decode_tc.cu): bfloat16, kv_rank up to 640, rot_dim up to 64.
bool latent_decode_tc_supported(const b200nn_ctx *ctx, const LatentDims &d);
size_t latent_decode_tc_part_floats(const b200nn_ctx *ctx, const LatentDims &d, int n_rows, int cap);
int launch_latent_decode_tc(b200nn_ctx *ctx, const LatentDims &d, const __nv_bfloat16 *q, const __nv_bfloat16 *qlat, const __nv_bfloat16 *cache,
                            int ring, size_t cache_rows, const RowMap &rows, int n_rows, int cap, __nv_bfloat16 *out, float *part);

// ---- gated delta rule ------------------------------------------------------------------------------
// Projection rows (f32): [q kv_heads*dim_p | k kv_heads*dim_p | v heads*vdim_p | gate heads*vdim_p | b heads |
// a heads]; the first three sections pass the short convolution.
struct DeltaDims {
    int heads, kv_heads, dim, dim_p, vdim, vdim_p, taps;
    float eps;
    HD int q_at() const { return 0; }
    HD int k_at() const { return kv_heads * dim_p; }
    HD int v_at() const { return 2 * kv_heads * dim_p; }
    HD int conv_w() const { return 2 * kv_heads * dim_p + heads * vdim_p; }
    HD int g_at() const { return conv_w(); }
    HD int b_at() const { return g_at() + heads * vdim_p; }
    HD int a_at() const { return b_at() + heads; }
    HD int proj_w() const { return (b_at() + 2 * heads + 3) & ~3; } // rows keep 16-byte alignment
    // convolved rows of a prompt pass (delta_rule.cu)
    HD int decay_at() const { return conv_w(); }
    HD int beta_at() const { return conv_w() + heads; }
    HD int kq_at() const { return conv_w() + 2 * heads; }
    HD int conv_ld() const { return (conv_w() + 2 * heads + kv_heads + 3) & ~3; }
};
struct DeltaWeights {
    const float *conv;    // [taps][conv_w]
    const float *a_exp;   // exp(A_log) [heads]
    const float *dt_bias; // [heads]
    const float *norm;    // [vdim]
};
// One token of every row: convolution, unit norms, decay, state update, read-out, output norm and gate.
int launch_delta_step(b200nn_ctx *ctx, const DeltaDims &d, bool b16, const float *proj, int ldp, const DeltaWeights &w, float *conv_state,
                      float *state, const RowMap &rows, int n_rows, void *out);
// Prompt rows.  conv: [n_rows][conv_ld] f32 scratch, heads_out:
// [n_rows][heads*vdim_p] f32 read-outs before their norm.
int launch_delta_prompt(b200nn_ctx *ctx, const DeltaDims &d, bool b16, const float *proj, int ldp, const DeltaWeights &w,
                        float *conv_state, float *state, const RowMap &rows, const SeqMap &sm, int n_rows, const int *row_seq, float *conv,
                        float *heads_out, void *out);

// ---- small pieces (kernels_elementwise.cu) -------------------------------------------------------------
int launch_rmsnorm(b200nn_ctx *ctx, const float *x, const float *w, float eps, int rows, int d, int ldo, void *out, int out_type);
int launch_embedding_rows(b200nn_ctx *ctx, const uint32_t *ids, const void *table, bool b16, int ldt, int n_rows, int d, int vocab,
                          float *out);
int launch_glu(b200nn_ctx *ctx, const float *gu, int rows, int n2, int act, float *out); // [rows][n2] quads -> [rows][n2/2]
int launch_gather_rows(b200nn_ctx *ctx, const float *src, const int *idx, int n_rows, int d, float *dst);
// y[m, g*out_stride + n] = sum_k x[m*ldx + g*x_stride + k] * w[g][n][k] (f32), times the epilogue's row scale
int launch_grouped_f32(b200nn_ctx *ctx, const float *w, int groups, int Ng, int Kg, const float *x, int ldx, int x_stride, int M,
                       const Epilogue &epi, int out_stride);
