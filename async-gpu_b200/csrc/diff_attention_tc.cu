#include "hybrid.h"
bool diff_prefill_tc_supported(const b200nn_ctx *, const DiffDims &) { return false; }
int launch_diff_prefill_tc(b200nn_ctx *ctx, const DiffDims &d, const __nv_bfloat16 *q, int ldq, const __nv_bfloat16 *cache, int cap, size_t cache_rows,
                           const SeqMap &sm, int n_rows, const float *gate, int gate_ld, __nv_bfloat16 *out) { return 1; }
bool diff_decode_tc_supported(const b200nn_ctx *, const DiffDims &) { return false; }
size_t diff_decode_tc_part_floats(const b200nn_ctx *ctx, const DiffDims &d, int n_rows, int cap) { return 0; }
int launch_diff_decode_tc(b200nn_ctx *ctx, const DiffDims &d, const __nv_bfloat16 *q, int ldq, const __nv_bfloat16 *cache, int cap, size_t cache_rows,
                          const RowMap &rows, int n_rows, const float *gate, int gate_ld, float *part, __nv_bfloat16 *out) { return 1; }
