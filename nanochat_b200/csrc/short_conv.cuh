/*
 * A short causal convolution over time on every projected channel (ncb_conv in include/nanochat_b200.h), as device functions
 * of the mixers that read projected rows: y_t = sum_j w[j] u_(t - taps + 1 + j), zeros before the sequence's start. The taps
 * before a pass's first row of a sequence come from a ring per slot that keeps the projected value of position p at p % taps.
 */
#pragma once

#include "ncb_common.cuh"

namespace {

template <typename T> __device__ __forceinline__ float to_f(T v) { return (float)v; }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16_rn(v); }

/* Two neighbouring values as one load and store. */
template <typename T> __device__ __forceinline__ float2 load2(const T *p);
template <> __device__ __forceinline__ float2 load2<float>(const float *p) { return *reinterpret_cast<const float2 *>(p); }
template <> __device__ __forceinline__ float2 load2<bf16>(const bf16 *p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(p)); }
__device__ __forceinline__ void store2(float *p, float x, float y) { *reinterpret_cast<float2 *>(p) = make_float2(x, y); }
__device__ __forceinline__ void store2(bf16 *p, float x, float y) { *reinterpret_cast<__nv_bfloat162 *>(p) = __floats2bfloat162_rn(x, y); }

/* Where a row stands: its position and slot, and how many rows just before it in the pass (at most taps - 1) are its
 * sequence's previous positions. */
struct Place {
    int pos, slot, before;
};
__device__ __forceinline__ Place place_of(const ncb_conv &c, int row) {
    Place p = {c.pos[row], c.slot_map ? c.slot_map[row] : row, 0};
    while (p.before < c.taps - 1) {
        const int r = row - p.before - 1;
        if (r < 0 || c.pos[r] != p.pos - p.before - 1 || (c.slot_map ? c.slot_map[r] : r) != p.slot || c.pos[r] < 0) break;
        p.before++;
    }
    return p;
}
constexpr int CONV_BATCH = 4; /* taps whose loads are in flight together */

/* Channels ch, ch + 1 (ch even) of row `row` after the convolution. */
template <typename T> __device__ __forceinline__ float2 conv2(const ncb_conv &c, int row, const Place &at, int ch) {
    const T *u = (const T *)c.proj + (size_t)row * c.ldp + ch;
    const T *ring = (const T *)c.ring + (size_t)at.slot * c.taps * c.width + ch;
    const int here = at.pos % c.taps;
    float2 y = make_float2(0.f, 0.f);
    for (int back0 = 0; back0 < c.taps; back0 += CONV_BATCH) {
        float2 w[CONV_BATCH], x[CONV_BATCH];
#pragma unroll
        for (int i = 0; i < CONV_BATCH; i++) {
            const int back = back0 + i;
            w[i] = x[i] = make_float2(0.f, 0.f);
            if (back < c.taps && back <= at.pos) {
                w[i] = *reinterpret_cast<const float2 *>(c.w + (size_t)(c.taps - 1 - back) * c.width + ch);
                x[i] = load2<T>(back <= at.before ? u - (ptrdiff_t)back * c.ldp : ring + (size_t)(here - back + (here < back ? c.taps : 0)) * c.width);
            }
        }
#pragma unroll
        for (int i = 0; i < CONV_BATCH; i++) y.x = fmaf(w[i].x, x[i].x, y.x), y.y = fmaf(w[i].y, x[i].y, y.y);
    }
    return y;
}
/* Four neighbouring values. */
__device__ __forceinline__ float4 load4(const float *p) { return *reinterpret_cast<const float4 *>(p); }
__device__ __forceinline__ float4 load4(const bf16 *p) {
    const uint2 v = *reinterpret_cast<const uint2 *>(p);
    return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16), __uint_as_float(v.y & 0xffff0000u));
}
__device__ __forceinline__ void store4(float *p, float4 v) { *reinterpret_cast<float4 *>(p) = v; }
__device__ __forceinline__ void store4(bf16 *p, float4 v) {
    uint2 o;
    reinterpret_cast<__nv_bfloat162 &>(o.x) = __floats2bfloat162_rn(v.x, v.y);
    reinterpret_cast<__nv_bfloat162 &>(o.y) = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2 *>(p) = o;
}
/* Keeps channels ch, ch + 1 of the row in the ring. A row on its own may do so at once: it reads the other taps' places. */
template <typename T> __device__ __forceinline__ void keep2(const ncb_conv &c, int row, const Place &at, int ch) {
    const float2 v = load2<T>((const T *)c.proj + (size_t)row * c.ldp + ch);
    store2((T *)c.ring + ((size_t)at.slot * c.taps + at.pos % c.taps) * c.width + ch, v.x, v.y);
}

inline int check_conv(const ncb_conv &c) {
    if (c.rows < 0 || c.rows > 0x7fffff00LL || c.taps < 1 || c.taps > 64 || c.width <= 0 || c.width % 8 || c.n_slots <= 0 || c.ldp < c.width || c.ldp % 2) return NCB_ERR_ARG;
    if (c.rows == 0) return NCB_OK;
    if (!c.proj || !c.ring || !c.w || !c.pos) return NCB_ERR_ARG;
    return ((uintptr_t)c.proj | (uintptr_t)c.ring | (uintptr_t)c.w) % 16 ? NCB_ERR_ALIGN : NCB_OK;
}

/* A launch with programmatic stream serialisation, in clusters of `cluster` blocks along x. */
template <typename... A>
int launch(void (*kernel)(A...), dim3 grid, int threads, size_t smem, int cluster, cudaStream_t stream, A... args) {
    if (smem > 48 * 1024 && cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
        return NCB_ERR_LAUNCH;
    cudaLaunchConfig_t config = {};
    config.gridDim = grid;
    config.blockDim = dim3(threads);
    config.dynamicSmemBytes = smem;
    config.stream = stream;
    cudaLaunchAttribute attribute[2];
    attribute[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attribute[0].val.programmaticStreamSerializationAllowed = 1;
    attribute[1].id = cudaLaunchAttributeClusterDimension;
    attribute[1].val.clusterDim.x = cluster;
    attribute[1].val.clusterDim.y = 1;
    attribute[1].val.clusterDim.z = 1;
    config.attrs = attribute;
    config.numAttrs = 2;
    return cudaLaunchKernelEx(&config, kernel, args...) == cudaSuccess ? NCB_OK : NCB_ERR_LAUNCH;
}

} /* namespace */
