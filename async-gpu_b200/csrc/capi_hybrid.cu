// The hybrid decoders' sequence mechanisms as stand-alone, stream-ordered operations on caller-owned device
// buffers (the kernels the model path launches).
#include "hybrid.h"

namespace {

bool latent_dims(const b200nn_latent_shape *s, LatentDims *d) {
    for (int v : {s->heads, s->dim, s->rot_dim, s->vdim, s->kv_rank})
        if (v <= 0) return false;
    if ((s->dim | s->rot_dim | s->vdim | s->kv_rank) & 15 || s->window < 0) return false;
    *d = LatentDims{s->heads, s->dim, s->rot_dim, s->rot_dim, s->vdim, s->kv_rank, s->kv_rank, 0, 0, s->window, s->scale, 0.0f};
    return true;
}

bool delta_dims(const b200nn_delta_shape *s, DeltaDims *d) {
    for (int v : {s->heads, s->kv_heads, s->dim, s->vdim, s->conv})
        if (v <= 0) return false;
    if ((s->dim | s->vdim) & 15 || s->heads % s->kv_heads) return false;
    *d = DeltaDims{s->heads, s->kv_heads, s->dim, s->dim, s->vdim, s->vdim, s->conv, s->eps};
    return true;
}

bool unaligned(std::initializer_list<const void *> ps) {
    for (const void *p : ps)
        if (!p || ((uintptr_t)p & 15)) return true;
    return false;
}

}  // namespace

extern "C" int32_t b200nn_latent_prefill_attention(b200nn_ctx *ctx, const b200nn_latent_shape *shape, uint32_t flags, const void *q_dev,
                                                   const void *kv_dev, const void *latent_dev, const float *gate_dev, int32_t n_rows,
                                                   int32_t k_rows, int32_t n_seq, int32_t max_n, const int32_t *seq_dev, void *out_dev) {
    LatentDims d;
    if (!ctx || !shape || !seq_dev || !gate_dev || n_rows <= 0 || k_rows <= 0 || n_seq <= 0 || max_n <= 0) return B200NN_ERR_ARG;
    if (!latent_dims(shape, &d)) return set_error(ctx, B200NN_ERR_SHAPE, "latent attention: sizes must be positive multiples of 16");
    if (unaligned({q_dev, kv_dev, latent_dev, out_dev})) return set_error(ctx, B200NN_ERR_ARG, "latent attention: buffers must be 16-byte aligned");
    CK(ctx, cudaSetDevice(ctx->device));
    SeqMap sm;
    sm.n_seq = n_seq;
    sm.max_n = max_n;
    sm.k_rows = k_rows;
    sm.row0 = seq_dev;
    sm.n = seq_dev + n_seq;
    sm.past = seq_dev + 2 * n_seq;
    sm.krow0 = seq_dev + 3 * n_seq;
    sm.kpos0 = seq_dev + 4 * n_seq;
    return launch_latent_prefill(ctx, d, !(flags & B200NN_LM_F32), n_rows, q_dev, kv_dev, latent_dev, sm, gate_dev, out_dev);
}

extern "C" int32_t b200nn_latent_decode_attention(b200nn_ctx *ctx, const b200nn_latent_shape *shape, uint32_t flags, const void *q_dev,
                                                  const void *qlat_dev, const void *cache_dev, int32_t ring, const int32_t *pos_dev,
                                                  const int32_t *slot_dev, int32_t n_slots, int32_t n_rows, int32_t capacity, void *out_dev) {
    LatentDims d;
    if (!ctx || !shape || !pos_dev || n_rows <= 0 || n_slots <= 0 || ring <= 0 || capacity <= 0) return B200NN_ERR_ARG;
    if (!latent_dims(shape, &d)) return set_error(ctx, B200NN_ERR_SHAPE, "latent attention: sizes must be positive multiples of 16");
    if (ring % 128 || (d.window ? ring < d.window : ring < capacity))
        return set_error(ctx, B200NN_ERR_SHAPE, "latent attention: the ring must be a multiple of 128 rows and hold the window");
    if (unaligned({q_dev, qlat_dev, cache_dev, out_dev})) return set_error(ctx, B200NN_ERR_ARG, "latent attention: buffers must be 16-byte aligned");
    CK(ctx, cudaSetDevice(ctx->device));
    const size_t need = latent_decode_part_floats(ctx, d, !(flags & B200NN_LM_F32), n_rows, capacity) * sizeof(float);
    if (need) TRY(ensure_scratch(ctx, need, 0));
    return launch_latent_decode(ctx, d, !(flags & B200NN_LM_F32), q_dev, qlat_dev, cache_dev, ring, (size_t)n_slots * ring, RowMap{pos_dev, 1, slot_dev}, n_rows, capacity,
                                out_dev, ctx->scratch);
}

static int delta_rule(b200nn_ctx *ctx, const DeltaDims &d, uint32_t flags, const float *proj_dev, const float *ext_dev, const b200nn_delta_weights *w,
                      float *conv_state_dev, float *state_dev, const int32_t *pos_dev, const int32_t *slot_dev, int32_t n_rows, int32_t n_seq,
                      int32_t max_n, const int32_t *seq_dev, float *scratch_dev, void *out_dev) {
    if (unaligned({proj_dev, conv_state_dev, state_dev, out_dev})) return set_error(ctx, B200NN_ERR_ARG, "delta rule: buffers must be 16-byte aligned");
    CK(ctx, cudaSetDevice(ctx->device));
    const DeltaWeights dw{w->conv, w->a_exp, w->dt_bias, w->norm};
    const bool b16 = !(flags & B200NN_LM_F32);
    const RowMap rows{pos_dev, 1, slot_dev};
    if (n_seq == 0) return launch_delta_step(ctx, d, b16, proj_dev, d.proj_w(), ext_dev, dw, conv_state_dev, state_dev, rows, n_rows, out_dev);
    if (!seq_dev || !slot_dev || max_n <= 0 || unaligned({scratch_dev})) return B200NN_ERR_ARG;
    SeqMap sm;
    sm.n_seq = n_seq;
    sm.max_n = max_n;
    sm.slot = seq_dev;
    sm.row0 = seq_dev + n_seq;
    sm.n = seq_dev + 2 * n_seq;
    sm.past = seq_dev + 3 * n_seq;
    return launch_delta_prompt(ctx, d, b16, proj_dev, d.proj_w(), ext_dev, dw, conv_state_dev, state_dev, rows, sm, n_rows, seq_dev + 4 * n_seq,
                               scratch_dev, scratch_dev + (size_t)n_rows * d.conv_ld(), out_dev);
}

extern "C" int32_t b200nn_delta_rule(b200nn_ctx *ctx, const b200nn_delta_shape *shape, uint32_t flags, const float *proj_dev,
                                     const b200nn_delta_weights *w, float *conv_state_dev, float *state_dev, const int32_t *pos_dev,
                                     const int32_t *slot_dev, int32_t n_rows, int32_t n_seq, int32_t max_n, const int32_t *seq_dev,
                                     float *scratch_dev, void *out_dev) {
    DeltaDims d;
    if (!ctx || !shape || !w || !pos_dev || n_rows <= 0 || n_seq < 0 || !w->conv || !w->a_exp || !w->dt_bias || !w->norm) return B200NN_ERR_ARG;
    if (!delta_dims(shape, &d)) return set_error(ctx, B200NN_ERR_SHAPE, "delta rule: dim and vdim must be positive multiples of 16");
    return delta_rule(ctx, d, flags, proj_dev, nullptr, w, conv_state_dev, state_dev, pos_dev, slot_dev, n_rows, n_seq, max_n, seq_dev, scratch_dev,
                      out_dev);
}

extern "C" int32_t b200nn_channel_delta_rule(b200nn_ctx *ctx, const b200nn_delta_shape *shape, uint32_t flags, const float *proj_dev,
                                             const float *ext_dev, const b200nn_delta_weights *w, float *conv_state_dev,
                                             float *state_dev, const int32_t *pos_dev, const int32_t *slot_dev, int32_t n_rows,
                                             int32_t n_seq, int32_t max_n, const int32_t *seq_dev, float *scratch_dev, void *out_dev) {
    DeltaDims d;
    if (!ctx || !shape || !w || !pos_dev || n_rows <= 0 || n_seq < 0 || !w->conv || !w->a_exp || !w->dt_bias || !w->norm) return B200NN_ERR_ARG;
    if (!delta_dims(shape, &d)) return set_error(ctx, B200NN_ERR_SHAPE, "delta rule: dim and vdim must be positive multiples of 16");
    if (unaligned({ext_dev})) return set_error(ctx, B200NN_ERR_ARG, "delta rule: buffers must be 16-byte aligned");
    d.channel = 1;
    return delta_rule(ctx, d, flags, proj_dev, ext_dev, w, conv_state_dev, state_dev, pos_dev, slot_dev, n_rows, n_seq, max_n, seq_dev, scratch_dev,
                      out_dev);
}

extern "C" int32_t b200nn_mlstm(b200nn_ctx *ctx, const b200nn_mlstm_shape *shape, uint32_t flags, const float *proj_dev,
                                const b200nn_mlstm_weights *w, float *memory_dev, float *normaliser_dev, float *maximum_dev,
                                const int32_t *pos_dev, const int32_t *slot_dev, int32_t n_rows, int32_t n_seq, const int32_t *seq_dev,
                                float *scratch_dev, void *out_dev) {
    if (!ctx || !shape || !w || !pos_dev || n_rows <= 0 || n_seq < 0 || !w->i_bias || !w->f_bias || !w->norm) return B200NN_ERR_ARG;
    const b200nn_mlstm_shape &s = *shape;
    if (s.heads <= 0 || s.dim <= 0 || s.vdim <= 0 || (s.dim | s.vdim) & 15 || !(s.gate_cap > 0.0f))
        return set_error(ctx, B200NN_ERR_SHAPE, "mlstm: dim and vdim must be positive multiples of 16, gate_cap positive");
    if (unaligned({proj_dev, memory_dev, normaliser_dev, out_dev}) || !maximum_dev)
        return set_error(ctx, B200NN_ERR_ARG, "mlstm: buffers must be 16-byte aligned");
    CK(ctx, cudaSetDevice(ctx->device));
    const MlstmDims d{s.heads, s.dim, s.dim, s.vdim, s.vdim, s.gate_cap, s.eps};
    const MlstmWeights mw{w->i_bias, w->f_bias, w->norm};
    const MlstmState st{memory_dev, normaliser_dev, maximum_dev};
    const bool b16 = !(flags & B200NN_LM_F32);
    if (n_seq == 0) return launch_mlstm_step(ctx, d, b16, proj_dev, d.proj_w(), mw, st, RowMap{pos_dev, 1, slot_dev}, n_rows, out_dev);
    if (!seq_dev || unaligned({scratch_dev})) return B200NN_ERR_ARG;
    SeqMap sm;
    sm.n_seq = n_seq;
    sm.slot = seq_dev;
    sm.row0 = seq_dev + n_seq;
    sm.n = seq_dev + 2 * n_seq;
    sm.past = seq_dev + 3 * n_seq;
    return launch_mlstm_prompt(ctx, d, b16, proj_dev, d.proj_w(), mw, st, sm, n_rows, scratch_dev, scratch_dev + (size_t)n_rows * s.heads * 4, out_dev);
}

extern "C" int32_t b200nn_diff_attention(b200nn_ctx *ctx, const b200nn_diff_shape *shape, uint32_t flags, const void *q_dev,
                                         const void *cache_dev, int32_t capacity, int32_t n_slots, const int32_t *pos_dev,
                                         const int32_t *slot_dev, const float *gate_dev, int32_t n_rows, int32_t n_seq, int32_t max_n,
                                         const int32_t *seq_dev, void *out_dev) {
    if (!ctx || !shape || !pos_dev || !gate_dev || n_rows <= 0 || n_seq < 0 || capacity <= 0 || n_slots <= 0) return B200NN_ERR_ARG;
    const b200nn_diff_shape &s = *shape;
    if (s.heads <= 0 || s.kv_heads <= 0 || s.dim <= 0 || s.vdim <= 0 || (s.dim | s.vdim) & 15 || s.heads % s.kv_heads || s.temp_every <= 0)
        return set_error(ctx, B200NN_ERR_SHAPE, "differential attention: dim and vdim must be positive multiples of 16, heads a multiple of kv_heads");
    if (unaligned({q_dev, cache_dev, out_dev})) return set_error(ctx, B200NN_ERR_ARG, "differential attention: buffers must be 16-byte aligned");
    if (n_seq && (!seq_dev || max_n <= 0)) return B200NN_ERR_ARG;
    CK(ctx, cudaSetDevice(ctx->device));
    const DiffDims d{s.heads, s.kv_heads, s.dim, s.vdim, s.vdim, s.temp_every, s.scale, s.softcap, s.temp_coef, s.lam, s.diff, s.eps};
    const bool b16 = !(flags & B200NN_LM_F32);
    SeqMap sm;
    if (n_seq) {
        sm.n_seq = n_seq;
        sm.max_n = max_n;
        sm.slot = seq_dev;
        sm.row0 = seq_dev + n_seq;
        sm.n = seq_dev + 2 * n_seq;
        sm.past = seq_dev + 3 * n_seq;
    }
    const size_t need = n_seq ? 0 : diff_part_floats(ctx, d, b16, n_rows, capacity) * sizeof(float);
    if (need) TRY(ensure_scratch(ctx, need, 0));
    return launch_diff_attention(ctx, d, b16, q_dev, d.q_w(), cache_dev, capacity, (size_t)n_slots * s.kv_heads * capacity, RowMap{pos_dev, 1, slot_dev},
                                 sm, n_rows, gate_dev, s.heads, ctx->scratch, out_dev);
}

extern "C" int32_t b200nn_stream_step(b200nn_ctx *ctx, uint32_t flags, int32_t n_rows, int32_t streams, int32_t width, float *xs_dev,
                                      const float *x0_dev, const float *y_dev, const float *prev_dev, const float *next_dev,
                                      const float *norm_dev, float eps, void *out_dev, float *sum_out_dev) {
    if (!ctx || n_rows <= 0 || streams <= 0 || width <= 0 || (!x0_dev && !y_dev) || (y_dev && !prev_dev) || (!sum_out_dev && (!next_dev || !norm_dev)))
        return B200NN_ERR_ARG;
    if (unaligned({xs_dev, sum_out_dev ? sum_out_dev : out_dev}) || ((uintptr_t)x0_dev | (uintptr_t)y_dev | (uintptr_t)norm_dev) & 15)
        return set_error(ctx, B200NN_ERR_ARG, "residual streams: buffers must be 16-byte aligned");
    CK(ctx, cudaSetDevice(ctx->device));
    auto coef = [&](const float *p) { return p ? StreamCoef{p, p + streams, p + 2 * streams} : StreamCoef{nullptr, nullptr, nullptr}; };
    return launch_stream_step(ctx, StreamStep{n_rows, streams, width, width, xs_dev, x0_dev, y_dev, coef(prev_dev), coef(next_dev), norm_dev, eps, out_dev,
                                              sum_out_dev}, !(flags & B200NN_LM_F32));
}
