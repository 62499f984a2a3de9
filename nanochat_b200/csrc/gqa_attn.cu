/*
 * Softmax attention of grouped query heads over a cache of normed, rotated keys and plain values, for heads of any size:
 *     q, k = rms_norm(rotate(conv(W h))),  v = conv(W h),  out_h = sigmoid(g_h) softmax(q_h . k scale) v.
 * The short convolution runs over time on every channel (short_conv.cuh), the rotation turns a head's first `rot` dimensions,
 * the norm has no weight. A layer may read another layer's cache (own_kv 0): then it only prepares its queries.
 *
 * Cache: T [n_slots][kv_heads][capacity][dim + vdim], T = bf16 (float for a model that runs in 32-bit).
 *   - k_gqa_rows: convolution, rotation, norm; queries to a buffer, keys and values to the cache;
 *   - k_gqa_split_any, k_gqa_merge: split over positions in plain fp32 arithmetic, any sizes and T, then the merge of the
 *     chunks' un-normalised states (m in log2 units, l, o) and the gate.
 */
#include "short_conv.cuh"

namespace {

constexpr float LOG2E = 1.4426950408889634f;
constexpr int THREADS = 128;
constexpr int TILE = NCB_GQA_TILE;
constexpr int STATE_PAD = 4; /* floats in front of a state's o: m, l, 2 pad */

/* Tiles of a row's positions and how they are cut: shared by the split kernels and the merge. */
struct Cut {
    int len, tiles, n_chunks, per;
};
__device__ __forceinline__ Cut cut_of(int len, int chunk_tiles) {
    Cut c;
    c.len = len;
    c.tiles = (len + TILE - 1) / TILE;
    c.n_chunks = (c.tiles + chunk_tiles - 1) / chunk_tiles;
    c.per = c.n_chunks > 0 ? (c.tiles + c.n_chunks - 1) / c.n_chunks : 0;
    return c;
}
/* The row's attended length: 0 for an idle row (negative position) and for one outside the cache (flagged). */
__device__ __forceinline__ int length_of(const ncb_gqa &a, int row, int &slot) {
    const int pos = a.conv.pos[row];
    slot = a.conv.slot_map ? a.conv.slot_map[row] : row;
    if (pos < 0) return 0;
    if (pos >= a.capacity || pos >= a.table_len || slot < 0 || slot >= a.conv.n_slots) {
        flag(a.status, NCB_DEV_BAD_POSITION);
        return 0;
    }
    return pos + 1;
}
template <typename T> __device__ __forceinline__ T *cache_row(const ncb_gqa &a, int slot, int kv_head, int pos) {
    return (T *)a.kv + (((size_t)slot * a.kv_heads + kv_head) * a.capacity + pos) * (a.dim + a.vdim);
}

/* ---- queries, keys and values of a row -------------------------------------------------------------------------------- */

/* One warp: the convolved channels ch0 .. of a query or key head in `x` [dim] (shared memory), then rotated and normed to `out`. */
template <typename T> __device__ __forceinline__ void head_row(const ncb_gqa &a, int row, const Place &at, int ch0, float *x, T *out, int lane) {
    for (int i = 2 * lane; i < a.dim; i += 64) {
        *reinterpret_cast<float2 *>(x + i) = conv2<T>(a.conv, row, at, ch0 + i);
        if (a.keep) keep2<T>(a.conv, row, at, ch0 + i);
    }
    __syncwarp();
    const int half = a.rot / 2;
    const float *cs = a.cos + (size_t)at.pos * half, *sn = a.sin + (size_t)at.pos * half;
    float sum = 0.f;
    for (int i = lane; i < half; i += 32) { /* in place: a pair belongs to one lane */
        const float u = x[i], v = x[i + half], c = cs[i], s = sn[i];
        x[i] = u * c - v * s;
        x[i + half] = v * c + u * s;
    }
    __syncwarp();
    for (int i = lane; i < a.dim; i += 32) sum = fmaf(x[i], x[i], sum);
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    const float r = 1.f / sqrtf(sum / (float)a.norm_count + a.eps);
    for (int i = 2 * lane; i < a.dim; i += 64) store2(out + i, x[i] * r, x[i + 1] * r);
}

/* Grid (units / 4 rounded up, rows), a warp per unit of a row: the query heads, then with own_kv the key and the value heads.
 * q NULL: the query heads only keep their ring. */
template <typename T> __global__ void __launch_bounds__(THREADS) k_gqa_rows(const ncb_gqa a) {
    extern __shared__ float sm[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, unit = blockIdx.x * (THREADS / 32) + warp, row = blockIdx.y;
    const int H = a.heads, G = a.own_kv ? a.kv_heads : 0;
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    if (unit >= H + 2 * G) return;
    int slot;
    const int len = length_of(a, row, slot);
    if (len == 0) return;
    const Place at = place_of(a.conv, row);
    float *x = sm + warp * a.dim;
    if (unit < H) {
        if (a.q) head_row<T>(a, row, at, a.off_q + unit * a.dim, x, (T *)a.q + ((size_t)row * H + unit) * a.dim, lane);
        else if (a.keep)
            for (int i = 2 * lane; i < a.dim; i += 64) keep2<T>(a.conv, row, at, a.off_q + unit * a.dim + i);
    } else if (unit < H + G) {
        head_row<T>(a, row, at, a.off_k + (unit - H) * a.dim, x, cache_row<T>(a, slot, unit - H, len - 1), lane);
    } else {
        const int g = unit - H - G, ch0 = a.off_v + g * a.vdim;
        T *out = cache_row<T>(a, slot, g, len - 1) + a.dim;
        for (int i = 2 * lane; i < a.vdim; i += 64) {
            const float2 v = conv2<T>(a.conv, row, at, ch0 + i);
            store2(out + i, v.x, v.y);
            if (a.keep) keep2<T>(a.conv, row, at, ch0 + i);
        }
    }
}

/* ---- split over positions --------------------------------------------------------------------------------------------- */

/* Plain fp32 arithmetic: grid (max chunks, heads, rows), any sizes. */
constexpr int ANY_TILE = 128;
template <typename T> __global__ void __launch_bounds__(THREADS) k_gqa_split_any(const ncb_gqa a) {
    extern __shared__ float sm[]; /* q [dim], o [vdim], probabilities [ANY_TILE], reduction [8] */
    const int tid = threadIdx.x, row = blockIdx.z, h = blockIdx.y, W = a.dim + a.vdim;
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    int slot;
    const Cut cut = cut_of(length_of(a, row, slot), a.chunk_tiles);
    const int p0 = min((int)blockIdx.x * cut.per, cut.tiles) * TILE, p1 = min(min((int)(blockIdx.x + 1) * cut.per, cut.tiles) * TILE, cut.len);
    if (blockIdx.x >= cut.n_chunks || p0 >= p1) return;
    float *q = sm, *o = q + a.dim, *p = o + a.vdim, *red = p + ANY_TILE;
    const T *qr = (const T *)a.q + ((size_t)row * a.heads + h) * a.dim;
    for (int i = tid; i < a.dim; i += THREADS) q[i] = to_f(qr[i]);
    for (int i = tid; i < a.vdim; i += THREADS) o[i] = 0.f;
    __syncthreads();
    const T *cache = cache_row<T>(a, slot, h / (a.heads / a.kv_heads), 0);
    float m = -INFINITY, l = 0.f;
    for (int at = p0; at < p1; at += ANY_TILE) {
        const int n = min(ANY_TILE, p1 - at);
        float s = -INFINITY;
        if (tid < n) {
            const T *c = cache + (size_t)(at + tid) * W;
            float v = 0.f;
            for (int i = 0; i < a.dim; i += 2) {
                const float2 k = load2<T>(c + i);
                v = fmaf(q[i], k.x, fmaf(q[i + 1], k.y, v));
            }
            s = v * a.scale * LOG2E;
        }
        float mx = s;
        for (int w = 16; w > 0; w >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, w));
        if ((tid & 31) == 0) red[tid >> 5] = mx;
        __syncthreads();
        mx = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
        const float next = fmaxf(m, mx), shrink = exp2f(m - next), e = exp2f(s - next);
        p[tid] = e;
        float sum = e;
        for (int w = 16; w > 0; w >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, w);
        if ((tid & 31) == 0) red[4 + (tid >> 5)] = sum;
        __syncthreads();
        l = l * shrink + ((red[4] + red[5]) + (red[6] + red[7]));
        m = next;
        for (int i = tid; i < a.vdim; i += THREADS) {
            float v = o[i] * shrink;
            for (int j = 0; j < n; j++) v = fmaf(p[j], to_f(cache[(size_t)(at + j) * W + a.dim + i]), v);
            o[i] = v;
        }
        __syncthreads();
    }
    float *out = a.parts + (((size_t)row * a.heads + h) * gridDim.x + blockIdx.x) * (a.vdim + STATE_PAD);
    if (tid == 0) out[0] = m, out[1] = l;
    for (int i = tid; i < a.vdim; i += THREADS) out[STATE_PAD + i] = o[i];
}

/* ---- merge and gate --------------------------------------------------------------------------------------------------- */

/* Grid (heads, rows): the chunks' states of a head, its gate. */
template <typename T> __global__ void __launch_bounds__(THREADS) k_gqa_merge(const ncb_gqa a) {
    extern __shared__ float w[]; /* factors [max_chunks] */
    const int tid = threadIdx.x, lane = tid & 31, h = blockIdx.x, row = blockIdx.y;
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    int slot;
    const int n = cut_of(length_of(a, row, slot), a.chunk_tiles).n_chunks;
    const size_t state = (size_t)(a.vdim + STATE_PAD);
    const float *p = a.parts + ((size_t)row * a.heads + h) * a.max_chunks * state;
    if (tid < 32) { /* the factor of chunk c's state: 2^(m_c - M) / L, times the gate */
        float M = -INFINITY, L = 0.f;
        for (int c = lane; c < n; c += 32) M = fmaxf(M, p[c * state]);
        for (int o = 16; o > 0; o >>= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, o));
        for (int c = lane; c < n; c += 32) {
            const float e = exp2f(p[c * state] - M);
            w[c] = e;
            L = fmaf(e, p[c * state + 1], L);
        }
        for (int o = 16; o > 0; o >>= 1) L += __shfl_xor_sync(0xffffffffu, L, o);
        const float z = to_f(((const T *)a.conv.proj)[(size_t)row * a.conv.ldp + a.off_g + h]);
        const float f = n > 0 ? 1.f / ((1.f + expf(-z)) * L) : 0.f;
        for (int c = lane; c < n; c += 32) w[c] *= f;
    }
    __syncthreads();
    T *out = (T *)a.out + (size_t)row * a.ldo + h * a.vdim;
    for (int i = 2 * tid; i < a.vdim; i += 2 * THREADS) {
        float2 v = make_float2(0.f, 0.f);
#pragma unroll 8
        for (int c = 0; c < n; c++) {
            const float2 s = *reinterpret_cast<const float2 *>(p + c * state + STATE_PAD + i);
            v.x = fmaf(w[c], s.x, v.x), v.y = fmaf(w[c], s.y, v.y);
        }
        store2(out + i, v.x, v.y);
    }
}

/* ---- host side -------------------------------------------------------------------------------------------------------- */

int check(const ncb_gqa &g) {
    const int rc = check_conv(g.conv);
    if (rc != NCB_OK || g.conv.rows == 0) return rc;
    if (g.conv.rows > 65535 * 64LL || g.heads <= 0 || g.kv_heads <= 0 || g.heads % g.kv_heads || g.heads > 65535 || g.dim <= 0 || g.dim % 16 ||
        g.vdim <= 0 || g.vdim % 16 || g.norm_count <= 0 || g.norm_count > g.dim || g.rot < 0 || g.rot % 2 || g.rot > g.dim || g.capacity <= 0 ||
        g.table_len <= 0)
        return NCB_ERR_ARG;
    const int W = g.conv.width;
    if (g.off_q < 0 || g.off_q % 2 || g.off_q + g.heads * g.dim > W || g.off_g < 0 || g.off_g + g.heads > g.conv.ldp) return NCB_ERR_ARG;
    if (g.own_kv && (g.off_k < 0 || g.off_k % 2 || g.off_k + g.kv_heads * g.dim > W || g.off_v < 0 || g.off_v % 2 || g.off_v + g.kv_heads * g.vdim > W))
        return NCB_ERR_ARG;
    if (!g.kv || (g.rot && (!g.cos || !g.sin))) return NCB_ERR_ARG;
    return ((uintptr_t)g.q | (uintptr_t)g.kv | (uintptr_t)g.parts | (uintptr_t)g.out) % 16 || g.ldo % 2 ? NCB_ERR_ALIGN : NCB_OK;
}
int check_parts(const ncb_gqa &g) {
    if (!g.q || !g.parts || g.chunk_tiles <= 0 || g.max_chunks <= 0 || g.max_len <= 0 || g.conv.rows > 65535 ||
        (long long)g.max_chunks * g.chunk_tiles * TILE < g.max_len)
        return NCB_ERR_ARG;
    return NCB_OK;
}

} /* namespace */

extern "C" {

int gqa_rows(const ncb_gqa *g, int f32, void *stream) {
    if (!g) return NCB_ERR_ARG;
    const int rc = check(*g);
    if (rc != NCB_OK || g->conv.rows == 0) return rc;
    if (g->conv.rows > 65535) return NCB_ERR_ARG;
    const size_t smem = (size_t)(THREADS / 32) * g->dim * 4;
    if (smem > 200 * 1024) return NCB_ERR_UNSUPPORTED;
    const int units = g->heads + (g->own_kv ? 2 * g->kv_heads : 0);
    const dim3 grid((units + THREADS / 32 - 1) / (THREADS / 32), (unsigned)g->conv.rows);
    return f32 ? launch(k_gqa_rows<float>, grid, THREADS, smem, 1, (cudaStream_t)stream, *g)
               : launch(k_gqa_rows<bf16>, grid, THREADS, smem, 1, (cudaStream_t)stream, *g);
}

int gqa_split(const ncb_gqa *g, int f32, void *stream) {
    if (!g) return NCB_ERR_ARG;
    int rc = check(*g);
    if (rc != NCB_OK || g->conv.rows == 0) return rc;
    if ((rc = check_parts(*g)) != NCB_OK) return rc;
    const size_t smem = (size_t)(g->dim + g->vdim + ANY_TILE + 8) * 4;
    if (smem > 200 * 1024) return NCB_ERR_UNSUPPORTED;
    const dim3 grid(g->max_chunks, g->heads, (unsigned)g->conv.rows);
    return f32 ? launch(k_gqa_split_any<float>, grid, THREADS, smem, 1, (cudaStream_t)stream, *g)
               : launch(k_gqa_split_any<bf16>, grid, THREADS, smem, 1, (cudaStream_t)stream, *g);
}

int gqa_merge(const ncb_gqa *g, int f32, void *stream) {
    if (!g) return NCB_ERR_ARG;
    int rc = check(*g);
    if (rc != NCB_OK || g->conv.rows == 0) return rc;
    if ((rc = check_parts(*g)) != NCB_OK) return rc;
    if (!g->out || g->ldo < g->heads * g->vdim) return NCB_ERR_ARG;
    const size_t smem = (size_t)g->max_chunks * 4;
    if (smem > 200 * 1024) return NCB_ERR_UNSUPPORTED;
    const dim3 grid(g->heads, (unsigned)g->conv.rows);
    return f32 ? launch(k_gqa_merge<float>, grid, THREADS, smem, 1, (cudaStream_t)stream, *g)
               : launch(k_gqa_merge<bf16>, grid, THREADS, smem, 1, (cudaStream_t)stream, *g);
}

} /* extern "C" */
