// Pieces of the decode-attention kernels whose MMA rows are keys (latent_decode_tc.cu, diff_decode_tc.cu): four softmax
// warps (128 threads, one key each) that share maxima and sums of every column.
#pragma once
#include "tc_ptx.cuh"

namespace tc {

// Butterfly over the warp that also transposes: on return v[0] of lane l holds the reduction over all lanes of
// column l (N = 32) or l >> 1 (N = 16).
template <int N, bool MAX>
__device__ __forceinline__ void reduce_columns(float (&v)[N]) {
    const int lane = threadIdx.x & 31;
    int o = 16;
#pragma unroll
    for (int w = N / 2; w >= 1; w >>= 1, o >>= 1) {
        const bool up = (lane & o) != 0;
#pragma unroll
        for (int i = 0; i < w; ++i) {
            const float send = up ? v[i] : v[i + w], keep = up ? v[i + w] : v[i];
            const float r = __shfl_xor_sync(0xffffffffu, send, o);
            v[i] = MAX ? fmaxf(keep, r) : keep + r;
        }
    }
    if (N == 16) {
        const float r = __shfl_xor_sync(0xffffffffu, v[0], 1);
        v[0] = MAX ? fmaxf(v[0], r) : v[0] + r;
    }
}

__device__ __forceinline__ void bar_softmax() { asm volatile("bar.sync 1, 128;" ::: "memory"); }
// The same with a vote: every thread learns whether any of them wants to give up.
__device__ __forceinline__ bool bar_softmax_any(bool pred) {
    uint32_t r;
    asm volatile(
        "{\n\t.reg .pred p, q;\n\t"
        "setp.ne.u32 q, %1, 0;\n\t"
        "bar.red.or.pred p, 1, 128, q;\n\t"
        "selp.u32 %0, 1, 0, p;\n\t}"
        : "=r"(r)
        : "r"((uint32_t)pred)
        : "memory");
    return r != 0;
}

template <int N>
__device__ __forceinline__ void tmem_ld_cols(uint32_t addr, float (&f)[N]) {
#pragma unroll
    for (int c = 0; c < N; c += 16) {
        uint32_t v[16];
        tmem_ld_x16(addr + c, v);
#pragma unroll
        for (int i = 0; i < 16; ++i) f[c + i] = __uint_as_float(v[i]);
    }
}

}  // namespace tc
