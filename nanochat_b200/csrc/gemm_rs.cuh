/*
 * Shared by the GEMM libraries: what a GEMM does when it reads or writes a residual stream that is kept in fp32
 * (ncb_gemm_rs in include/nanochat_b200.h). Device side: the row scale that stands for an RMS norm of the input, the
 * stream update, the gated unit's activation. Host side: the checks of an ncb_gemm_rs.
 */
#pragma once

#include "ncb_common.cuh"

#include <type_traits>

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
    int streams; /* several streams: how they are read and written (ncb_gemm_rs epilogue 7) */
    float in[NCB_MAX_STREAMS], out[NCB_MAX_STREAMS], mix[NCB_MAX_STREAMS * NCB_MAX_STREAMS];
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

__device__ __forceinline__ float silu(float z) { return z / (1.f + expf(-z)); }
template <bool SILU> __device__ __forceinline__ float gate_of(float z) { return SILU ? silu(z) : gelu_tanh(z); }

__device__ __forceinline__ float axpy(float c, float x, float y) { return fmaf(c, x, y); }
__device__ __forceinline__ float4 axpy(float c, float4 x, float4 y) {
    return make_float4(fmaf(c, x.x, y.x), fmaf(c, x.y, y.y), fmaf(c, x.z, y.z), fmaf(c, x.w, y.w));
}
__device__ __forceinline__ float scaled(float c, float x) { return c * x; }
__device__ __forceinline__ float4 scaled(float c, float4 x) { return make_float4(c * x.x, c * x.y, c * x.z, c * x.w); }

/* The values of at most S streams in one place (a column, or four): `at` is the place's offset in the first stream, the
 * streams lie `stride` apart. update() writes every stream and returns what the next branch reads. */
template <int S, typename V> struct Streams {
    V h[S];
    __device__ __forceinline__ void load(const StreamIO &r, size_t at, int stride, bool on) {
#pragma unroll
        for (int s = 0; s < S; s++)
            h[s] = on && s < r.streams ? *reinterpret_cast<const V *>(r.h + at + (size_t)s * stride) : V{};
    }
    __device__ __forceinline__ V update(const StreamIO &r, size_t at, int stride, V v, bool on) const {
        V u = V{};
#pragma unroll
        for (int t = 0; t < S; t++) {
            V n = scaled(r.out[t], v);
#pragma unroll
            for (int s = 0; s < S; s++) n = axpy(r.mix[s * NCB_MAX_STREAMS + t], h[s], n);
            if (on && t < r.streams) *reinterpret_cast<V *>(r.h + at + (size_t)t * stride) = n;
            u = axpy(r.in[t], n, u);
        }
        return u;
    }
};
/* f(std::integral_constant<int, S>) with the smallest instantiated S that holds the streams. */
template <typename F> __device__ __forceinline__ void with_streams(int streams, F f) {
    if (streams <= 2) f(std::integral_constant<int, 2>());
    else if (streams <= 4) f(std::integral_constant<int, 4>());
    else f(std::integral_constant<int, NCB_MAX_STREAMS>());
}
/* One column of a row: load, update, the value the next branch reads. */
__device__ __forceinline__ float streams_add(const StreamIO &r, size_t row, int n, int N, float v) {
    float u = 0.f;
    with_streams(r.streams, [&](auto S) {
        Streams<decltype(S)::value, float> x;
        const size_t at = row * r.streams * N + n;
        x.load(r, at, N, true);
        u = x.update(r, at, N, v, true);
    });
    return u;
}

inline StreamIO no_stream() {
    StreamIO r = {};
    r.scale = 1.f;
    return r;
}

inline StreamIO stream_io(const ncb_gemm_rs &g) {
    StreamIO r = {g.ss, g.ss_parts, g.norm_count > 0 ? 1.f / (float)g.norm_count : 0.f, g.eps, g.scale,
                  g.h,  g.gain,     g.x_next,                                          g.ss_next, g.mult};
    if (g.epilogue != 7) return r;
    r.streams = g.streams;
    for (int s = 0; s < g.streams; s++) {
        r.in[s] = g.in[s], r.out[s] = g.out[s];
        for (int t = 0; t < g.streams; t++) r.mix[s * NCB_MAX_STREAMS + t] = g.mix[s * NCB_MAX_STREAMS + t];
    }
    return r;
}

inline int check_rs(const ncb_gemm_rs &g) {
    if (g.rows < 0 || g.N <= 0 || g.K <= 0) return NCB_ERR_ARG;
    if (g.epilogue != 0 && g.epilogue != 3 && (g.epilogue < 5 || g.epilogue > 8)) return NCB_ERR_ARG;
    if (g.epilogue == 7 && (g.streams < 1 || g.streams > NCB_MAX_STREAMS)) return NCB_ERR_ARG;
    if (g.rows == 0) return NCB_OK;
    if (!g.x || !g.w) return NCB_ERR_ARG;
    if (g.ss && (g.ss_parts <= 0 || g.norm_count <= 0)) return NCB_ERR_ARG;
    if ((uintptr_t)g.ss % 16) return NCB_ERR_ALIGN;
    if (g.epilogue == 6 || g.epilogue == 7) {
        if (!g.h || !g.gain || !g.x_next || !g.ss_next) return NCB_ERR_ARG;
        if (((uintptr_t)g.h | (uintptr_t)g.gain | (uintptr_t)g.x_next) % 16) return NCB_ERR_ALIGN;
    } else {
        const int columns = g.epilogue == 5 || g.epilogue == 8 ? g.N / 2 : g.n_store;
        if (!g.y || columns < 0 || columns > g.N || g.ldy < columns) return NCB_ERR_ARG;
        if ((uintptr_t)g.y % 16) return NCB_ERR_ALIGN;
    }
    return ((uintptr_t)g.x | (uintptr_t)g.w) % 16 ? NCB_ERR_ALIGN : NCB_OK;
}

} /* namespace */
