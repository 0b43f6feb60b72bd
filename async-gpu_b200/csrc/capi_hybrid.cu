// The hybrid decoder's sequence mechanisms as stand-alone, stream-ordered operations on caller-owned device
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

extern "C" int32_t b200nn_delta_rule(b200nn_ctx *ctx, const b200nn_delta_shape *shape, uint32_t flags, const float *proj_dev,
                                     const b200nn_delta_weights *w, float *conv_state_dev, float *state_dev, const int32_t *pos_dev,
                                     const int32_t *slot_dev, int32_t n_rows, int32_t n_seq, int32_t max_n, const int32_t *seq_dev,
                                     float *scratch_dev, void *out_dev) {
    DeltaDims d;
    if (!ctx || !shape || !w || !pos_dev || n_rows <= 0 || !w->conv || !w->a_exp || !w->dt_bias || !w->norm) return B200NN_ERR_ARG;
    if (!delta_dims(shape, &d)) return set_error(ctx, B200NN_ERR_SHAPE, "delta rule: dim and vdim must be positive multiples of 16");
    if (unaligned({proj_dev, conv_state_dev, state_dev, out_dev})) return set_error(ctx, B200NN_ERR_ARG, "delta rule: buffers must be 16-byte aligned");
    CK(ctx, cudaSetDevice(ctx->device));
    const DeltaWeights dw{w->conv, w->a_exp, w->dt_bias, w->norm};
    const bool b16 = !(flags & B200NN_LM_F32);
    const RowMap rows{pos_dev, 1, slot_dev};
    if (n_seq == 0) return launch_delta_step(ctx, d, b16, proj_dev, d.proj_w(), nullptr, dw, conv_state_dev, state_dev, rows, n_rows, out_dev);
    if (!seq_dev || !slot_dev || max_n <= 0 || unaligned({scratch_dev})) return B200NN_ERR_ARG;
    SeqMap sm;
    sm.n_seq = n_seq;
    sm.max_n = max_n;
    sm.slot = seq_dev;
    sm.row0 = seq_dev + n_seq;
    sm.n = seq_dev + 2 * n_seq;
    sm.past = seq_dev + 3 * n_seq;
    return launch_delta_prompt(ctx, d, b16, proj_dev, d.proj_w(), nullptr, dw, conv_state_dev, state_dev, rows, sm, n_rows, seq_dev + 4 * n_seq, scratch_dev,
                               scratch_dev + (size_t)n_rows * d.conv_ld(), out_dev);
}
