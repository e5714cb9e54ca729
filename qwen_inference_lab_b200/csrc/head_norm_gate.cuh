// What finishes the outputs of a recurrence with a state matrix per head: every head's e values divided by their own root
// mean square, times a weight of e that all heads share (null: none), times silu of a gate (null: none), float32 arithmetic.
#pragma once
#include "common.cuh"

// `nb` rows of one head in shared or global memory, `o_stride` apart, a warp per row; the gate and the result are rows of all
// heads (head h at column h * e) from token `first_token` on.
template <typename T, typename W>
__device__ __forceinline__ void head_norm_gate_rows(const float* o_rows, int o_stride, int nb, size_t first_token,
                                                    const T* g, int ld, const W* norm_w, float eps, int n_heads,
                                                    int head, int e, T* out, int lane, int warp, int warps) {
    for (int tb = warp; tb < nb; tb += warps) {
        const float* o = o_rows + (size_t)tb * o_stride;
        float ss = 0.f;
        for (int c = lane; c < e; c += 32) ss = fmaf(o[c], o[c], ss);
        ss = warp_sum(ss);
        const float scale = 1.0f / sqrtf(ss / (float)e + eps);
        const size_t token = first_token + tb;
        for (int c = lane; c < e; c += 32) {
            float y = o[c] * scale;
            if (norm_w != nullptr) y *= to_f32<W>(norm_w[c]);
            if (g != nullptr) {
                const float gate = to_f32<T>(g[token * ld + head * e + c]);
                y *= gate / (1.f + expf(-gate));
            }
            out[(token * n_heads + head) * e + c] = from_f32<T>(y);
        }
    }
}
