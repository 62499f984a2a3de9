/*
 * Shared by the GEMM libraries: what a GEMM does when it reads or writes a residual stream that is kept in fp32
 * (ncb_gemm_rs in include/nanochat_b200.h). Device side: the row scale that stands for an RMS norm of the input, the
 * stream update, the gated unit's activation. Host side: the checks of an ncb_gemm_rs.
 */
#pragma once

#include "ncb_common.cuh"

namespace {

struct StreamIO {
    const float *ss;
    int ss_parts;
    float inv_count, eps, scale;
    float *h;
    const float *gain;
    void *x_next;
    float *ss_next;
    float mult;
};

/* The factor of a row's product: scale, times 1 / rms of the stream row whose squares sum to `sum` when it is normed. */
__device__ __forceinline__ float row_scale(const StreamIO &r, float sum) {
    return r.ss ? r.scale * (1.f / sqrtf(sum * r.inv_count + r.eps)) : r.scale;
}
/* h[at] += mult * v; the new value. */
__device__ __forceinline__ float stream_add(const StreamIO &r, size_t at, float v) {
    const float h = r.h[at] + r.mult * v;
    r.h[at] = h;
    return h;
}
/* 0.5 z (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3))) */
__device__ __forceinline__ float gelu_tanh(float z) {
    return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

inline StreamIO no_stream() { return {nullptr, 0, 0.f, 0.f, 1.f, nullptr, nullptr, nullptr, nullptr, 0.f}; }

inline StreamIO stream_io(const ncb_gemm_rs &g) {
    return {g.ss, g.ss_parts, g.norm_count > 0 ? 1.f / (float)g.norm_count : 0.f, g.eps, g.scale,
            g.h,  g.gain,     g.x_next,                                          g.ss_next, g.mult};
}

inline int check_rs(const ncb_gemm_rs &g) {
    if (g.rows < 0 || g.N <= 0 || g.K <= 0) return NCB_ERR_ARG;
    if (g.epilogue != 0 && g.epilogue != 3 && g.epilogue != 5 && g.epilogue != 6) return NCB_ERR_ARG;
    if (g.rows == 0) return NCB_OK;
    if (!g.x || !g.w) return NCB_ERR_ARG;
    if (g.ss && (g.ss_parts <= 0 || g.norm_count <= 0)) return NCB_ERR_ARG;
    if ((uintptr_t)g.ss % 16) return NCB_ERR_ALIGN;
    if (g.epilogue == 6) {
        if (!g.h || !g.gain || !g.x_next || !g.ss_next) return NCB_ERR_ARG;
        if (((uintptr_t)g.h | (uintptr_t)g.gain | (uintptr_t)g.x_next) % 16) return NCB_ERR_ALIGN;
    } else {
        const int columns = g.epilogue == 5 ? g.N / 2 : g.n_store;
        if (!g.y || columns < 0 || columns > g.N || g.ldy < columns) return NCB_ERR_ARG;
        if ((uintptr_t)g.y % 16) return NCB_ERR_ALIGN;
    }
    return ((uintptr_t)g.x | (uintptr_t)g.w) % 16 ? NCB_ERR_ALIGN : NCB_OK;
}

} /* namespace */
