// Layer mechanisms of the hybrid decoders (hybrid.cu): gated delta rule with a decay per head or per key channel,
// matrix memory with exponential gates (mLSTM), latent attention, differential attention, residual streams.
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
// With `channel` the decay is one per head and key channel and the output gate a sigmoid instead of a silu; the inputs
// of both come from a two-step projection, rows of their own [decay inputs heads*dim_p .. | gate inputs heads*vdim_p ..],
// the two parts `ext` columns each.  The projection row is then [q | k | v | b | first step of the two, `low` columns each].
struct DeltaDims {
    int heads, kv_heads, dim, dim_p, vdim, vdim_p, taps;
    float eps;
    int channel = 0, low = 0;
    HD int q_at() const { return 0; }
    HD int k_at() const { return kv_heads * dim_p; }
    HD int v_at() const { return 2 * kv_heads * dim_p; }
    HD int conv_w() const { return 2 * kv_heads * dim_p + heads * vdim_p; }
    HD int g_at() const { return conv_w(); }
    HD int b_at() const { return channel ? conv_w() : g_at() + heads * vdim_p; }
    HD int a_at() const { return b_at() + heads; }
    HD int low_at() const { return (b_at() + heads + 15) & ~15; } // channel
    HD int ext() const { return heads * (dim_p > vdim_p ? dim_p : vdim_p); }
    HD int proj_w() const { return channel ? low_at() + 2 * low : (b_at() + 2 * heads + 3) & ~3; } // rows keep 16-byte alignment
    // convolved rows of a prompt pass (delta_rule.cu)
    HD int decays() const { return channel ? heads * dim_p : heads; }
    HD int decay_at() const { return conv_w(); }
    HD int beta_at() const { return conv_w() + decays(); }
    HD int kq_at() const { return beta_at() + heads; }
    HD int conv_ld() const { return (kq_at() + kv_heads + 3) & ~3; }
};
struct DeltaWeights {
    const float *conv;    // [taps][conv_w]
    const float *a_exp;   // exp(A_log) [heads]
    const float *dt_bias; // [heads], or [heads][dim_p] with `channel`
    const float *norm;    // [vdim]
};
// One token of every row: convolution, unit norms, decay, state update, read-out, output norm and gate.
// ext (channel only): [n_rows][2 * d.ext()] f32.
int launch_delta_step(b200nn_ctx *ctx, const DeltaDims &d, bool b16, const float *proj, int ldp, const float *ext, const DeltaWeights &w, float *conv_state,
                      float *state, const RowMap &rows, int n_rows, void *out);
// Prompt rows.  conv: [n_rows][conv_ld] f32 scratch, heads_out:
// [n_rows][heads*vdim_p] f32 read-outs before their norm.
int launch_delta_prompt(b200nn_ctx *ctx, const DeltaDims &d, bool b16, const float *proj, int ldp, const float *ext, const DeltaWeights &w,
                        float *conv_state, float *state, const RowMap &rows, const SeqMap &sm, int n_rows, const int *row_seq, float *conv,
                        float *heads_out, void *out);

// ---- matrix memory with exponential gates (mlstm.cu) ------------------------------------------------
// Projection rows (f32): [q heads*dim_p | k heads*dim_p | v heads*vdim_p | gate heads*vdim_p | i heads | f heads].
struct MlstmDims {
    int heads, dim, dim_p, vdim, vdim_p;
    float cap, eps;
    HD int q_at() const { return 0; }
    HD int k_at() const { return heads * dim_p; }
    HD int v_at() const { return 2 * heads * dim_p; }
    HD int g_at() const { return v_at() + heads * vdim_p; }
    HD int i_at() const { return g_at() + heads * vdim_p; }
    HD int f_at() const { return i_at() + heads; }
    HD int proj_w() const { return (f_at() + heads + 3) & ~3; }
};
struct MlstmWeights {
    const float *i_bias, *f_bias; // [heads]
    const float *norm;            // [heads][vdim_p]
};
// Per slot: memory f32 [heads][dim_p][vdim_p], normaliser [heads][dim_p], running maximum [heads].
struct MlstmState {
    float *memory, *normaliser, *maximum;
};
// One token of every row.
int launch_mlstm_step(b200nn_ctx *ctx, const MlstmDims &d, bool b16, const float *proj, int ldp, const MlstmWeights &w, const MlstmState &st,
                      const RowMap &rows, int n_rows, void *out);
// Prompt rows.  gates: [n_rows][heads][4] f32 scratch, heads_out: [n_rows][heads*vdim_p] f32.
int launch_mlstm_prompt(b200nn_ctx *ctx, const MlstmDims &d, bool b16, const float *proj, int ldp, const MlstmWeights &w, const MlstmState &st,
                        const SeqMap &sm, int n_rows, float *gates, float *heads_out, void *out);

// ---- differential attention (diff_attention*.cu, diff_decode_tc.cu) ----------------------------------
// Two softmax maps per head over the same values, o = a1 - lambda a2, over its root mean square, times (1 - diff) and
// the head's gate.  Query head h uses key / value head h / (heads / kv_heads).
//   query      [row][head][2 maps][dim_p]                            rows ldq apart
//   cache      [slot][kv head][position][2 maps * dim_p | vdim_p]        kv_w columns
// Scores are (q . k) * scale * temperature(position), then cap * tanh(score / cap) (cap 0: none); temperature is
// 1 + qt_coef * ln(floor((position + 1) / qt_every) + 1).
struct DiffDims {
    int heads, kv_heads, dim_p, vdim, vdim_p, qt_every;
    float scale, cap, qt_coef, lambda, diff, eps;
    HD int group() const { return heads / kv_heads; }
    HD int q_w() const { return heads * 2 * dim_p; }
    HD int kv_w() const { return 2 * dim_p + vdim_p; }
    HD int cache_w() const { return kv_heads * kv_w(); }
    HD float score_scale(int pos) const {
        return qt_coef == 0.0f ? scale : scale * (1.0f + qt_coef * logf((float)((pos + 1) / qt_every) + 1.0f));
    }
};
// The rows' own keys and values are in the cache (cap positions per slot and head).  gate: [n_rows][gate_ld] f32 before
// the sigmoid; out [row][head][vdim_p].  n_seq of sm: 0 for one token per row (decoding), where `part` of
// diff_part_floats is scratch and cache_rows = slots * kv_heads * cap.
int launch_diff_attention(b200nn_ctx *ctx, const DiffDims &d, bool b16, const void *q, int ldq, const void *cache, int cap, size_t cache_rows,
                          const RowMap &rows, const SeqMap &sm, int n_rows, const float *gate, int gate_ld, float *part, void *out);
size_t diff_part_floats(const b200nn_ctx *ctx, const DiffDims &d, bool b16, int n_rows, int cap);
bool diff_prefill_tc_supported(const b200nn_ctx *ctx, const DiffDims &d);
int launch_diff_prefill_tc(b200nn_ctx *ctx, const DiffDims &d, const __nv_bfloat16 *q, int ldq, const __nv_bfloat16 *cache, int cap, size_t cache_rows,
                           const SeqMap &sm, int n_rows, const float *gate, int gate_ld, __nv_bfloat16 *out);
bool diff_decode_tc_supported(const b200nn_ctx *ctx, const DiffDims &d);
size_t diff_decode_tc_part_floats(const b200nn_ctx *ctx, const DiffDims &d, int n_rows, int cap);
int launch_diff_decode_tc(b200nn_ctx *ctx, const DiffDims &d, const __nv_bfloat16 *q, int ldq, const __nv_bfloat16 *cache, int cap, size_t cache_rows,
                          const RowMap &rows, int n_rows, const float *gate, int gate_ld, float *part, __nv_bfloat16 *out);
// f32 models: columns [at, at + cache_w) of the projection rows -> the cache rows of the tokens.
int launch_kv_store_f32(b200nn_ctx *ctx, const float *proj, int ldp, int at, int kv_heads, int kv_w, int cap, const RowMap &rows, int n_rows,
                        float *cache);

// ---- residual streams (streams.cu) ---------------------------------------------------------------------
constexpr int MAX_STREAMS = 8;
struct StreamCoef {
    const float *in, *out, *mix; // [n], [n], [n from][n to]
};
// y set: the sublayer before (its `out` and `mix` in prev) is added to the streams xs [rows][n][d]; y null: every stream
// starts as x0 [rows][d].  Then the next sublayer's input (its `in` in next) goes through the RMS norm to out [rows][ldo];
// or, with x_sum, only the sum of the streams is left there ([rows][d]).
struct StreamStep {
    int rows, n, d, ldo;
    float *xs;
    const float *x0, *y;
    StreamCoef prev, next;
    const float *norm;
    float eps;
    void *out;
    float *x_sum;
};
int launch_stream_step(b200nn_ctx *ctx, const StreamStep &a, bool b16);

// ---- small pieces (kernels_elementwise.cu) -------------------------------------------------------------
int launch_rmsnorm(b200nn_ctx *ctx, const float *x, const float *w, float eps, int rows, int d, int ldo, void *out, int out_type);
// pos_table (may be null): learned position vectors [max_pos][ldt], added.
int launch_embedding_rows(b200nn_ctx *ctx, const uint32_t *ids, const void *table, bool b16, int ldt, int n_rows, int d, int vocab,
                          const void *pos_table, int max_pos, const RowMap &rows, float *out);
int launch_glu(b200nn_ctx *ctx, const float *gu, int rows, int n2, int act, float *out); // [rows][n2] quads -> [rows][n2/2]
int launch_gather_rows(b200nn_ctx *ctx, const float *src, const int *idx, int n_rows, int d, float *dst);
// y[m, g*out_stride + n] = sum_k x[m*ldx + g*x_stride + k] * w[g][n][k] (f32), times the epilogue's row scale
int launch_grouped_f32(b200nn_ctx *ctx, const float *w, int groups, int Ng, int Kg, const float *x, int ldx, int x_stride, int M,
                       const Epilogue &epi, int out_stride);
