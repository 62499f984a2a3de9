/*
 * Softmax attention of grouped query heads over a cache of normed, rotated keys and plain values, for heads of any size:
 *     q, k = rms_norm(rotate(conv(W h))),  v = conv(W h),  out_h = sigmoid(g_h) softmax(q_h . k scale) v.
 * The short convolution runs over time on every channel (short_conv.cuh), the rotation turns a head's first `rot` dimensions,
 * the norm has no weight. A layer may read another layer's cache (own_kv 0): then it only prepares its queries.
 *
 * Cache: T [n_slots][kv_heads][capacity][dim + vdim], T = bf16 (float for a model that runs in 32-bit).
 *   - k_gqa_rows (prompts): convolution, rotation, norm; queries to a buffer, keys and values to the cache;
 *   - k_gqa_split (decode, short portions): split over positions, the query heads of one key/value head as the M of
 *     mma.sync.m16n8k16. Every warp walks its own 16-position tiles, whose rows come by bulk copies into its own ring, with a
 *     softmax state of its own; the block merges its four. In a decode step it also does what k_gqa_rows does: the copies of
 *     the older positions start before the dependency wait, and the new row goes to the cache and straight to its tile;
 *   - k_gqa_merge: the chunks' un-normalised states (m in log2 units, l, o) and the gate;
 *   - k_gqa_prefill: a tile of a prompt's rows of one query head against the cached keys and values.
 * Scores and probabilities are fp32; a probability enters the second product as two bf16 terms (hi + lo), so its weight keeps
 * 16 bits. k_gqa_split_any is the split in plain fp32 arithmetic for any sizes and for T = float.
 */
#include "short_conv.cuh"
#include "umma.cuh"

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

constexpr int RUN = 16; /* consecutive rows a warp of k_gqa_rows works on */

/* Shared memory per warp of k_gqa_rows: the projected rows with the taps before them, the convolution's weights (CONV_BATCH of
 * them, zero past the taps), two of a head's rows, the rows' places. */
__host__ __device__ inline size_t rows_smem(int size, int itemsize) {
    return (size_t)(RUN + CONV_BATCH - 1) * size * itemsize + (size_t)CONV_BATCH * size * 4 + (size_t)2 * size * 4 + RUN * sizeof(Place) + 8;
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void *src, bool on) { /* 16 bytes, zeros when off */
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(on ? 16 : 0) : "memory");
}

/* Grid (units / warps rounded up, rows / RUN rounded up), a warp per unit and run of rows: the query heads, then with own_kv the
 * key and the value heads. q NULL: the query heads only keep their ring. A loop over the rows with a short body: the kernel has
 * many warps, and what is unrolled far has to be fetched by each of them. */
template <typename T> __global__ void __launch_bounds__(THREADS, 7) k_gqa_rows(const ncb_gqa a) {
    extern __shared__ __align__(128) uint8_t raw[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, unit = blockIdx.x * (blockDim.x >> 5) + warp;
    const int H = a.heads, G = a.own_kv ? a.kv_heads : 0, row0 = blockIdx.y * RUN, n = (int)min((long long)RUN, a.conv.rows - row0);
    constexpr int OLD = CONV_BATCH - 1, PER = 16 / sizeof(T);
    const int largest = max(a.dim, a.vdim);
    uint8_t *mine = raw + warp * ((rows_smem(largest, sizeof(T)) + 15) / 16 * 16);
    T *tile = reinterpret_cast<T *>(mine);                                  /* [OLD + RUN][size] */
    float *w = reinterpret_cast<float *>(tile + (OLD + RUN) * largest);     /* [CONV_BATCH][size], by how far back */
    float *x = w + CONV_BATCH * largest;                                    /* [2][size] */
    Place *place = reinterpret_cast<Place *>(x + 2 * largest);
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    if (unit >= H + 2 * G) return;
    const bool query = unit < H, key = !query && unit < H + G;
    const int kvh = query ? 0 : key ? unit - H : unit - H - G, size = query || key ? a.dim : a.vdim;
    const int ch0 = query ? a.off_q + unit * a.dim : key ? a.off_k + kvh * a.dim : a.off_v + kvh * a.vdim;
    const T *proj = (const T *)a.conv.proj + ch0;
    const int per = size / PER, first = row0 - OLD;
#pragma unroll 4
    for (int i = lane; i < (OLD + n) * per; i += 32) {
        const int r = i / per, c = (i - r * per) * PER;
        cp_async16(smem_u32(tile + r * size + c), proj + (size_t)max(first + r, 0) * a.conv.ldp + c, first + r >= 0);
    }
    for (int i = lane; i < CONV_BATCH * size / 4; i += 32) {
        const int back = 4 * i / size, c = 4 * i - back * size;
        const bool on = back < a.conv.taps;
        cp_async16(smem_u32(w + 4 * i), a.conv.w + (size_t)(on ? a.conv.taps - 1 - back : 0) * a.conv.width + ch0 + c, on);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    bool elsewhere = false;
    if (lane < n) {
        int slot;
        const int len = length_of(a, row0 + lane, slot);
        const Place at = len ? place_of(a.conv, row0 + lane) : Place{-1, 0, 0};
        place[lane] = at;
        elsewhere = at.before < a.conv.taps - 1 || a.conv.taps > CONV_BATCH; /* some tap is not a row of the pass */
    }
    const uint32_t special = __ballot_sync(0xffffffffu, elsewhere);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncwarp();
    const int half = a.rot / 2;
    const float inv_count = 1.f / (float)a.norm_count;
    auto norm_scale = [&](float sum) { return sizeof(T) == 2 ? rsqrtf(fmaf(sum, inv_count, a.eps)) : 1.f / sqrtf(sum / (float)a.norm_count + a.eps); };
    if (a.keep)
        for (int r = 0; r < n; r++)
            if (place[r].pos >= 0)
                for (int i = 2 * lane; i < size; i += 64) keep2<T>(a.conv, row0 + r, place[r], ch0 + i);
    if (query && !a.q) return;
    if (size <= 128) { /* four channels per lane: two rows at a time, weights and older taps in registers */
        const int i = 4 * lane;
        const bool on = i < size;
        /* lane r: where row r goes (NULL: nowhere) and its position */
        int pos = -1;
        T *to = nullptr;
        if (lane < n) {
            const Place at = place[lane];
            pos = at.pos;
            if (pos >= 0) to = query ? (T *)a.q + ((size_t)(row0 + lane) * H + unit) * a.dim : cache_row<T>(a, at.slot, kvh, pos) + (key ? 0 : a.dim);
        }
        float4 f[CONV_BATCH], v[OLD + 2];
#pragma unroll
        for (int back = 0; back < CONV_BATCH; back++) f[back] = on ? load4(w + back * size + i) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int j = 0; j < OLD; j++) v[j] = on ? load4(tile + j * size + i) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 1
        for (int r = 0; r < n; r += 2) {
            T *out[2];
            float4 y[2];
#pragma unroll
            for (int e = 0; e < 2; e++) {
                out[e] = reinterpret_cast<T *>(__shfl_sync(0xffffffffu, reinterpret_cast<unsigned long long>(to), r + e));
                v[OLD + e] = on ? load4(tile + (min(r + e, n - 1) + OLD) * size + i) : make_float4(0.f, 0.f, 0.f, 0.f);
                y[e] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                for (int back = 0; back < CONV_BATCH; back++) {
                    const float4 c = f[back], u = v[OLD + e - back];
                    y[e].x = fmaf(c.x, u.x, y[e].x), y[e].y = fmaf(c.y, u.y, y[e].y), y[e].z = fmaf(c.z, u.z, y[e].z), y[e].w = fmaf(c.w, u.w, y[e].w);
                }
            }
#pragma unroll
            for (int j = 0; j < OLD; j++) v[j] = v[j + 2];
            if (special >> r & 3)
                for (int e = 0; e < 2; e++)
                    if ((special >> (r + e) & 1) && out[e] && on) {
                        const float2 lo = conv2<T>(a.conv, row0 + r + e, place[r + e], ch0 + i), hi = conv2<T>(a.conv, row0 + r + e, place[r + e], ch0 + i + 2);
                        const float4 z = make_float4(lo.x, lo.y, hi.x, hi.y);
                        if (e) y[1] = z;
                        else y[0] = z;
                    }
            if (!query && !key) {
#pragma unroll
                for (int e = 0; e < 2; e++)
                    if (out[e] && on) store4(out[e] + i, y[e]);
                continue;
            }
            if (half) {
                if (on) *reinterpret_cast<float4 *>(x + i) = y[0], *reinterpret_cast<float4 *>(x + size + i) = y[1];
                __syncwarp();
                const int p0 = max(__shfl_sync(0xffffffffu, pos, r), 0), p1 = max(__shfl_sync(0xffffffffu, pos, r + 1), 0);
                for (int j = lane; j < 2 * half; j += 32) { /* in place: a pair belongs to one lane */
                    const bool second = j >= half;
                    const int d = second ? j - half : j;
                    const size_t at = (size_t)(second ? p1 : p0) * half + d;
                    float *row = x + (second ? size : 0) + d;
                    const float c = a.cos[at], s = a.sin[at], u = row[0], z = row[half];
                    row[0] = u * c - z * s;
                    row[half] = z * c + u * s;
                }
                __syncwarp();
                if (on) y[0] = load4(x + i), y[1] = load4(x + size + i);
            }
            /* both rows' sums of squares in one reduction: a half of the warp each */
            float sq[2];
#pragma unroll
            for (int e = 0; e < 2; e++) sq[e] = fmaf(y[e].x, y[e].x, fmaf(y[e].y, y[e].y, fmaf(y[e].z, y[e].z, y[e].w * y[e].w)));
            float sum = (lane & 16 ? sq[1] : sq[0]) + __shfl_xor_sync(0xffffffffu, lane & 16 ? sq[0] : sq[1], 16);
#pragma unroll
            for (int o = 8; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
            const float scale = norm_scale(sum);
#pragma unroll
            for (int e = 0; e < 2; e++) {
                const float g = __shfl_sync(0xffffffffu, scale, 16 * e);
                if (out[e] && on) store4(out[e] + i, make_float4(y[e].x * g, y[e].y * g, y[e].z * g, y[e].w * g));
            }
        }
        return;
    }
#pragma unroll 1
    for (int r = 0; r < n; r++) {
        const Place at = place[r];
        if (at.pos < 0) continue;
        T *out = query ? (T *)a.q + ((size_t)(row0 + r) * H + unit) * a.dim : cache_row<T>(a, at.slot, kvh, at.pos) + (key ? 0 : a.dim);
        for (int i = 4 * lane; i < size; i += 128) {
            float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
            if (special >> r & 1) {
                const float2 u = conv2<T>(a.conv, row0 + r, at, ch0 + i), v = conv2<T>(a.conv, row0 + r, at, ch0 + i + 2);
                y = make_float4(u.x, u.y, v.x, v.y);
            } else {
#pragma unroll
                for (int back = 0; back < CONV_BATCH; back++) {
                    const float4 f = *reinterpret_cast<const float4 *>(w + back * size + i), v = load4(tile + (r + OLD - back) * size + i);
                    y.x = fmaf(f.x, v.x, y.x), y.y = fmaf(f.y, v.y, y.y), y.z = fmaf(f.z, v.z, y.z), y.w = fmaf(f.w, v.w, y.w);
                }
            }
            if (query || key) *reinterpret_cast<float4 *>(x + i) = y;
            else store4(out + i, y);
        }
        if (!query && !key) continue;
        __syncwarp();
        for (int i = lane; i < half; i += 32) { /* in place: a pair belongs to one lane */
            const float c = a.cos[(size_t)at.pos * half + i], s = a.sin[(size_t)at.pos * half + i], u = x[i], v = x[i + half];
            x[i] = u * c - v * s;
            x[i + half] = v * c + u * s;
        }
        __syncwarp();
        float sum = 0.f;
        for (int i = 4 * lane; i < size; i += 128) {
            const float4 v = *reinterpret_cast<const float4 *>(x + i);
            sum = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, sum))));
        }
        for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
        const float f = norm_scale(sum);
        for (int i = 4 * lane; i < size; i += 128) {
            const float4 v = *reinterpret_cast<const float4 *>(x + i);
            store4(out + i, make_float4(v.x * f, v.y * f, v.z * f, v.w * f));
        }
        __syncwarp();
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

__device__ __forceinline__ void mma_bf16(float *d, const uint32_t *a, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, "
                 "{%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm4(uint32_t *r, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4_t(uint32_t *r, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t *>(&v);
}
/* hi = bf16(v) and lo = bf16(v - hi) of two values. */
__device__ __forceinline__ void split_bf16(float x, float y, uint32_t &hi, uint32_t &lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const float2 f = __bfloat1622float2(h);
    hi = *reinterpret_cast<const uint32_t *>(&h);
    lo = pack_bf16(x - f.x, y - f.y);
}

constexpr int WARPS = THREADS / 32, HEADS_M = 16; /* query heads per block = MMA M */

/* Shared memory of k_gqa_split in bytes: the warps' rings (then their states), q, the new row, the warps' scratch, barriers. */
struct SplitSmem {
    int stage, q, row, scratch, bars, total;
};
__host__ __device__ inline SplitSmem split_smem(int dim, int vdim, int stages) {
    SplitSmem s;
    s.stage = TILE * ((dim + vdim) * 2 + 16);
    s.q = WARPS * stages * s.stage;
    s.row = s.q + HEADS_M * (dim + 8) * 2;
    s.scratch = s.row + (dim + vdim) * 2;
    s.bars = s.scratch + WARPS * dim * 4;
    s.total = s.bars + WARPS * stages * 8;
    return s;
}

/* Grid (max chunks, kv_heads x tiles of 16 query heads, rows). DK, VN: upper bounds of dim / 16 and vdim / 16. */
template <int DK, int VN> __global__ void __launch_bounds__(THREADS, DK + VN > 16 ? 1 : 2) k_gqa_split(const ncb_gqa a, int stages) {
    extern __shared__ __align__(128) uint8_t raw[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3, row = blockIdx.z;
    const int R = a.heads / a.kv_heads, head_tiles = (R + HEADS_M - 1) / HEADS_M, kvh = blockIdx.y / head_tiles;
    const int h0 = kvh * R + blockIdx.y % head_tiles * HEADS_M, n_heads = min(HEADS_M, (kvh + 1) * R - h0);
    const int W = a.dim + a.vdim, stride = W * 2 + 16;
    const SplitSmem L = split_smem(a.dim, a.vdim, stages);
    const uint32_t base = smem_u32(raw), ring = base + warp * stages * L.stage, bars = base + L.bars + warp * stages * 8;
    const bool fused = a.q == nullptr; /* a decode step: this launch prepares its row itself */
    if (lane < stages) mbar_init(bars + 8 * lane, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    __syncwarp();
    if (!fused) asm volatile("griddepcontrol.wait;" ::: "memory");
    int slot;
    const Cut cut = cut_of(length_of(a, row, slot), a.chunk_tiles);
    const int t0 = blockIdx.x * cut.per, t1 = min(t0 + cut.per, cut.tiles);
    const bool idle = blockIdx.x >= cut.n_chunks || t0 >= t1, last = t1 == cut.tiles;
    const int n_tiles = idle ? 0 : (t1 - t0 - warp + WARPS - 1) / WARPS; /* this warp's tiles: t0 + warp, + WARPS, .. */
    const int stored = cut.len - (fused && a.own_kv ? 1 : 0);            /* positions the cache holds already */
    const bf16 *cache = cache_row<bf16>(a, idle ? 0 : slot, kvh, 0);
    auto fetch = [&](int i) { /* the stored rows of tile i of this warp */
        const int s = i % stages, p0 = (t0 + warp + i * WARPS) * TILE, n = min(TILE, stored - p0);
        if (lane == 0) mbar_expect_tx(bars + 8 * s, (n > 0 ? n : 0) * W * 2);
        __syncwarp();
        if (lane < n) bulk_load(ring + s * L.stage + lane * stride, cache + (size_t)(p0 + lane) * W, W * 2, bars + 8 * s);
    };
    for (int i = 0; i < min(stages, n_tiles); i++) fetch(i);
    if (fused) asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    if (idle) return;
    bf16 *qs = reinterpret_cast<bf16 *>(raw + L.q), *fresh = reinterpret_cast<bf16 *>(raw + L.row);
    const int qstride = a.dim + 8;
    if (fused) {
        const Place at = place_of(a.conv, row);
        float *x = reinterpret_cast<float *>(raw + L.scratch) + warp * a.dim;
        ncb_gqa b = a; /* the rings are kept once: queries by the first chunk, key and value by the last */
        b.keep = a.keep && blockIdx.x == 0;
        for (int u = warp; u < n_heads; u += WARPS) {
            head_row<bf16>(b, row, at, a.off_q + (h0 + u) * a.dim, x, qs + u * qstride, lane);
            __syncwarp();
        }
        if (a.own_kv && last) {
            const bool first_tile = blockIdx.y % head_tiles == 0; /* of this key/value head: it alone writes */
            b.keep = a.keep && first_tile;
            if (warp == n_heads % WARPS) head_row<bf16>(b, row, at, a.off_k + kvh * a.dim, x, fresh, lane);
            if (warp == (n_heads + 1) % WARPS)
                for (int i = 2 * lane; i < a.vdim; i += 64) {
                    const float2 v = conv2<bf16>(a.conv, row, at, a.off_v + kvh * a.vdim + i);
                    store2(fresh + a.dim + i, v.x, v.y);
                    if (b.keep) keep2<bf16>(a.conv, row, at, a.off_v + kvh * a.vdim + i);
                }
        }
    } else {
        for (int i = tid; i < n_heads * (a.dim / 8); i += THREADS)
            *reinterpret_cast<uint4 *>(qs + i / (a.dim / 8) * qstride + i % (a.dim / 8) * 8) =
                *reinterpret_cast<const uint4 *>((const bf16 *)a.q + ((size_t)row * a.heads + h0) * a.dim + (size_t)i * 8);
    }
    for (int i = tid; i < (HEADS_M - n_heads) * (a.dim / 8); i += THREADS)
        *reinterpret_cast<uint4 *>(qs + (n_heads + i / (a.dim / 8)) * qstride + i % (a.dim / 8) * 8) = make_uint4(0u, 0u, 0u, 0u);
    __syncthreads();
    if (fused && a.own_kv && last && blockIdx.y % head_tiles == 0)
        for (int i = tid; i < W / 8; i += THREADS)
            *reinterpret_cast<uint4 *>((bf16 *)cache + (size_t)(cut.len - 1) * W + i * 8) = *reinterpret_cast<const uint4 *>(fresh + i * 8);
    const int dk = a.dim / 16, vn = a.vdim / 16;
    uint32_t qf[DK][4];
    {
        const uint32_t qa = base + L.q + ((lane & 15) * qstride + (lane >> 4) * 8) * 2;
#pragma unroll
        for (int k = 0; k < DK; k++)
            if (k < dk) ldsm4(qf[k], qa + k * 32);
    }
    float o[VN][2][4];
#pragma unroll
    for (int i = 0; i < VN; i++)
#pragma unroll
        for (int j = 0; j < 8; j++) o[i][j >> 2][j & 3] = 0.f;
    float m_lo = -INFINITY, m_hi = -INFINITY, l_lo = 0.f, l_hi = 0.f;
    const float scale = a.scale * LOG2E;
    bool ok = true;
    for (int i = 0; i < n_tiles; i++) {
        const int s = i % stages, p0 = (t0 + warp + i * WARPS) * TILE, live = min(TILE, cut.len - p0), there = max(0, min(TILE, stored - p0));
        const uint32_t stage = ring + s * L.stage;
        if (!mbar_wait(bars + 8 * s, (i / stages) & 1)) ok = false;
        __syncwarp();
        if (there < TILE) { /* the sequence's last tile: its new row, and zeros past its end */
            uint8_t *rows = raw + warp * stages * L.stage + s * L.stage;
            for (int j = lane; j < (TILE - there) * (W / 8); j += 32) {
                const int r = there + j / (W / 8), c = j % (W / 8);
                *reinterpret_cast<uint4 *>(rows + r * stride + c * 16) = r < live ? *reinterpret_cast<const uint4 *>(fresh + c * 8) : make_uint4(0u, 0u, 0u, 0u);
            }
            __syncwarp();
        }
        float p[2][4] = {};
        const uint32_t kb = stage + ((lane >> 4) * 8 + (lane & 7)) * stride + ((lane >> 3) & 1) * 16;
#pragma unroll
        for (int k = 0; k < DK; k++)
            if (k < dk) {
                uint32_t b[4];
                ldsm4(b, kb + k * 32);
                mma_bf16(p[0], qf[k], b[0], b[1]);
                mma_bf16(p[1], qf[k], b[2], b[3]);
            }
        float mx_lo = m_lo, mx_hi = m_hi;
#pragma unroll
        for (int n = 0; n < 2; n++)
#pragma unroll
            for (int e = 0; e < 2; e++) {
                const bool on = n * 8 + 2 * t + e < live;
                p[n][e] = on ? p[n][e] * scale : -INFINITY, p[n][2 + e] = on ? p[n][2 + e] * scale : -INFINITY;
                mx_lo = fmaxf(mx_lo, p[n][e]), mx_hi = fmaxf(mx_hi, p[n][2 + e]);
            }
        mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 1));
        mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 1));
        mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 2));
        mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 2));
        if (__any_sync(0xffffffffu, mx_lo != m_lo || mx_hi != m_hi)) {
            const float al = ex2(m_lo - mx_lo), ah = ex2(m_hi - mx_hi); /* 0 for the first tile */
            l_lo *= al, l_hi *= ah;
#pragma unroll
            for (int c = 0; c < VN; c++)
#pragma unroll
                for (int n = 0; n < 2; n++) o[c][n][0] *= al, o[c][n][1] *= al, o[c][n][2] *= ah, o[c][n][3] *= ah;
            m_lo = mx_lo, m_hi = mx_hi;
        }
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; e++) { /* e: heads g / g + 8, positions 2 t, + 1 / + 8, + 9 */
            const float m = (e & 1) ? m_hi : m_lo;
            const float a0 = ex2(p[e >> 1][2 * (e & 1)] - m), a1 = ex2(p[e >> 1][2 * (e & 1) + 1] - m);
            if (e & 1) l_hi += a0 + a1;
            else l_lo += a0 + a1;
            split_bf16(a0, a1, hi[e], lo[e]);
        }
        const uint32_t vb = stage + a.dim * 2 + (lane & 15) * stride + (lane >> 4) * 16;
#pragma unroll
        for (int c = 0; c < VN; c++)
            if (c < vn) {
                uint32_t b[4];
                ldsm4_t(b, vb + c * 32);
                mma_bf16(o[c][0], hi, b[0], b[1]);
                mma_bf16(o[c][1], hi, b[2], b[3]);
                mma_bf16(o[c][0], lo, b[0], b[1]);
                mma_bf16(o[c][1], lo, b[2], b[3]);
            }
        __syncwarp(); /* the stage may be overwritten */
        if (i + stages < n_tiles) fetch(i + stages);
    }
    if (!ok && lane == 0) flag(a.status, NCB_DEV_WAIT_TIMEOUT);
    l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 1);
    l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 1);
    l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 2);
    l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 2);
    __syncthreads(); /* every ring has been consumed: the warps' states take its place */
    const int state = a.vdim + STATE_PAD;
    float *mine = reinterpret_cast<float *>(raw) + warp * HEADS_M * state;
    if (t == 0) {
        mine[g * state] = m_lo, mine[g * state + 1] = l_lo;
        mine[(g + 8) * state] = m_hi, mine[(g + 8) * state + 1] = l_hi;
    }
#pragma unroll
    for (int c = 0; c < VN; c++)
        if (c < vn)
#pragma unroll
            for (int n = 0; n < 2; n++) {
                const int col = STATE_PAD + c * 16 + n * 8 + 2 * t;
                *reinterpret_cast<float2 *>(mine + g * state + col) = make_float2(o[c][n][0], o[c][n][1]);
                *reinterpret_cast<float2 *>(mine + (g + 8) * state + col) = make_float2(o[c][n][2], o[c][n][3]);
            }
    __syncthreads();
    for (int h = warp; h < n_heads; h += WARPS) { /* (the chunk's first tile is never empty: some m is finite) */
        const float *s = reinterpret_cast<const float *>(raw) + h * state;
        float M = -INFINITY, f[WARPS], l = 0.f;
#pragma unroll
        for (int w = 0; w < WARPS; w++) M = fmaxf(M, s[w * HEADS_M * state]);
#pragma unroll
        for (int w = 0; w < WARPS; w++) {
            f[w] = exp2f(s[w * HEADS_M * state] - M);
            l = fmaf(f[w], s[w * HEADS_M * state + 1], l);
        }
        float *out = a.parts + (((size_t)row * a.heads + h0 + h) * gridDim.x + blockIdx.x) * state;
        if (lane == 0) out[0] = M, out[1] = l;
        for (int i = STATE_PAD + 2 * lane; i < state; i += 64) {
            float2 v = make_float2(0.f, 0.f);
#pragma unroll
            for (int w = 0; w < WARPS; w++) {
                const float2 x = *reinterpret_cast<const float2 *>(s + w * HEADS_M * state + i);
                v.x = fmaf(f[w], x.x, v.x), v.y = fmaf(f[w], x.y, v.y);
            }
            *reinterpret_cast<float2 *>(out + i) = v;
        }
    }
}

/* ---- prompts ---------------------------------------------------------------------------------------------------------- */

constexpr int PF_ROWS = 64, PF_KEYS = 64; /* query rows and keys per tile: four warps of 16 rows */

/* Grid (heads, row tiles): at most PF_ROWS consecutive rows of one sequence, one query head. Keys and values of 64 positions
 * per stage (cp.async, two stages); a warp owns 16 rows over the whole range. QS, VN: upper bounds of dim / 16 and vdim / 16
 * (with EXACT the values). */
template <int QS, int VN, bool EXACT> __global__ void __launch_bounds__(THREADS, 2) k_gqa_prefill(const ncb_gqa a) {
    extern __shared__ __align__(128) uint8_t raw[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int h = blockIdx.x, tile = blockIdx.y, dim = EXACT ? QS * 16 : a.dim, vdim = EXACT ? VN * 16 : a.vdim;
    const int steps = dim / 16, cols = vdim / 16, W = dim + vdim, stride = W * 2 + 16, stage_bytes = PF_KEYS * stride;
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const int row0 = a.tile_row[tile], n_rows = min(a.tile_rows[tile], PF_ROWS), pos0 = a.tile_pos[tile];
    const int keys = pos0 + n_rows, n_tiles = (keys + PF_KEYS - 1) / PF_KEYS; /* the last row sees positions < keys */
    int slot;
    if (length_of(a, row0, slot) == 0 || length_of(a, row0 + n_rows - 1, slot) != keys) return; /* flagged by gqa_rows too */
    const uint32_t smem = smem_u32(raw);
    const bf16 *kv = cache_row<bf16>(a, slot, h / (a.heads / a.kv_heads), 0);
    auto fetch = [&](int i) {
        const uint32_t dst = smem + (i & 1) * stage_bytes;
        const int p0 = i * PF_KEYS, n = W / 8, c0 = tid & 7;
#pragma unroll
        for (int j = 0; j < PF_KEYS / 16; j++) { /* eight threads per row, 16 rows at a time */
            const int r = (tid >> 3) + 16 * j;
            const bool on = p0 + r < keys;
            const bf16 *src = kv + (size_t)(on ? p0 + r : 0) * W;
#pragma unroll(EXACT ? (QS + VN) * 2 / 8 : 1)
            for (int c = c0; c < n; c += 8) cp_async16(dst + r * stride + c * 16, src + c * 8, on);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(0);
    uint32_t qf[QS][4];
    const int lo_row = warp * 16 + g, hi_row = lo_row + 8;
    const bool lo_on = lo_row < n_rows, hi_on = hi_row < n_rows;
    {
        const bf16 *q = (const bf16 *)a.q + ((size_t)row0 * a.heads + h) * dim + 2 * t;
        const bf16 *lo = q + (size_t)lo_row * a.heads * dim, *hi = q + (size_t)hi_row * a.heads * dim;
#pragma unroll
        for (int i = 0; i < QS; i++) {
            const bool on = i < steps;
            qf[i][0] = on && lo_on ? *reinterpret_cast<const uint32_t *>(lo + i * 16) : 0u;
            qf[i][1] = on && hi_on ? *reinterpret_cast<const uint32_t *>(hi + i * 16) : 0u;
            qf[i][2] = on && lo_on ? *reinterpret_cast<const uint32_t *>(lo + i * 16 + 8) : 0u;
            qf[i][3] = on && hi_on ? *reinterpret_cast<const uint32_t *>(hi + i * 16 + 8) : 0u;
        }
    }
    float o[VN][2][4];
#pragma unroll
    for (int i = 0; i < VN; i++)
#pragma unroll
        for (int j = 0; j < 8; j++) o[i][j >> 2][j & 3] = 0.f;
    float m_lo = -INFINITY, m_hi = -INFINITY, l_lo = 0.f, l_hi = 0.f;
    const float scale = a.scale * LOG2E;
    const int lo_pos = pos0 + lo_row, hi_pos = pos0 + hi_row, warp_last = pos0 + warp * 16 + 15;
    for (int i = 0; i < n_tiles; i++) {
        if (i + 1 < n_tiles) {
            fetch(i + 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const uint32_t ks = smem + (i & 1) * stage_bytes, vs = ks + dim * 2;
        const int p0 = i * PF_KEYS;
        if (p0 <= warp_last) { /* some row of this warp sees some key of the tile */
            float s[PF_KEYS / 8][4];
#pragma unroll
            for (int n = 0; n < PF_KEYS / 8; n++) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
            const uint32_t kbase = ks + ((lane >> 4) * 8 + (lane & 7)) * stride + ((lane >> 3) & 1) * 16;
#pragma unroll
            for (int k = 0; k < QS; k++)
                if (k < steps) {
#pragma unroll
                    for (int n = 0; n < PF_KEYS / 16; n++) {
                        uint32_t b[4];
                        ldsm4(b, kbase + n * 16 * stride + k * 32);
                        mma_bf16(s[2 * n], qf[k], b[0], b[1]);
                        mma_bf16(s[2 * n + 1], qf[k], b[2], b[3]);
                    }
                }
            const bool edge = p0 + PF_KEYS - 1 > pos0 + warp * 16; /* the causal border crosses this tile */
            float mx_lo = m_lo, mx_hi = m_hi;
#pragma unroll
            for (int n = 0; n < PF_KEYS / 8; n++)
#pragma unroll
                for (int e = 0; e < 2; e++) {
                    const int p = p0 + n * 8 + 2 * t + e;
                    s[n][e] = edge && p > lo_pos ? -INFINITY : s[n][e] * scale;
                    s[n][2 + e] = edge && p > hi_pos ? -INFINITY : s[n][2 + e] * scale;
                    mx_lo = fmaxf(mx_lo, s[n][e]);
                    mx_hi = fmaxf(mx_hi, s[n][2 + e]);
                }
            mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 1));
            mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 2));
            mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 1));
            mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 2));
            /* position 0 is visible to every row and in the first tile, so the maxima are finite from there on */
            if (__any_sync(0xffffffffu, mx_lo != m_lo || mx_hi != m_hi)) {
                const float al = ex2(m_lo - mx_lo), ah = ex2(m_hi - mx_hi);
                l_lo *= al, l_hi *= ah;
#pragma unroll
                for (int c = 0; c < VN; c++)
#pragma unroll
                    for (int n = 0; n < 2; n++) o[c][n][0] *= al, o[c][n][1] *= al, o[c][n][2] *= ah, o[c][n][3] *= ah;
                m_lo = mx_lo, m_hi = mx_hi;
            }
            const uint32_t vbase = vs + (lane & 15) * stride + (lane >> 4) * 16;
#pragma unroll
            for (int j = 0; j < PF_KEYS / 16; j++) { /* 16 keys: two score tiles are one A operand */
                uint32_t hi[4], lo[4];
#pragma unroll
                for (int e = 0; e < 4; e++) { /* e: rows g / g + 8, keys 2 t, + 1 / + 8, + 9 */
                    const int n = 2 * j + (e >> 1);
                    const float m = (e & 1) ? m_hi : m_lo;
                    const float a0 = ex2(s[n][2 * (e & 1)] - m), a1 = ex2(s[n][2 * (e & 1) + 1] - m);
                    if (e & 1) l_hi += a0 + a1;
                    else l_lo += a0 + a1;
                    split_bf16(a0, a1, hi[e], lo[e]);
                }
#pragma unroll
                for (int c = 0; c < VN; c++)
                    if (c < cols) {
                        uint32_t b[4];
                        ldsm4_t(b, vbase + j * 16 * stride + c * 32);
                        mma_bf16(o[c][0], hi, b[0], b[1]);
                        mma_bf16(o[c][1], hi, b[2], b[3]);
                        mma_bf16(o[c][0], lo, b[0], b[1]);
                        mma_bf16(o[c][1], lo, b[2], b[3]);
                    }
            }
        }
        __syncthreads(); /* the stage may be overwritten */
    }
    l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 1);
    l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 2);
    l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 1);
    l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 2);
#pragma unroll
    for (int r = 0; r < 2; r++)
        if (r ? hi_on : lo_on) {
            const int row = row0 + (r ? hi_row : lo_row);
            const float z = to_f(((const bf16 *)a.conv.proj)[(size_t)row * a.conv.ldp + a.off_g + h]);
            const float f = 1.f / ((1.f + expf(-z)) * (r ? l_hi : l_lo));
            bf16 *out = (bf16 *)a.out + (size_t)row * a.ldo + h * vdim + 2 * t;
#pragma unroll
            for (int c = 0; c < VN; c++)
                if (c < cols)
#pragma unroll
                    for (int n = 0; n < 2; n++)
                        *reinterpret_cast<uint32_t *>(out + c * 16 + n * 8) = pack_bf16(o[c][n][2 * r] * f, o[c][n][2 * r + 1] * f);
        }
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
    if (g.off_q < 0 || g.off_q % 4 || g.off_q + g.heads * g.dim > W || g.off_g < 0 || g.off_g + g.heads > g.conv.ldp) return NCB_ERR_ARG;
    if (g.own_kv && (g.off_k < 0 || g.off_k % 4 || g.off_k + g.kv_heads * g.dim > W || g.off_v < 0 || g.off_v % 4 || g.off_v + g.kv_heads * g.vdim > W))
        return NCB_ERR_ARG;
    if (!g.kv || (g.rot && (!g.cos || !g.sin))) return NCB_ERR_ARG;
    return ((uintptr_t)g.q | (uintptr_t)g.kv | (uintptr_t)g.parts | (uintptr_t)g.out) % 16 || g.ldo % 2 || g.conv.ldp % 4 ? NCB_ERR_ALIGN : NCB_OK;
}
int check_parts(const ncb_gqa &g) {
    if (!g.parts || g.chunk_tiles <= 0 || g.max_chunks <= 0 || g.max_len <= 0 || g.conv.rows > 65535 ||
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
    const size_t one = (rows_smem(g->dim > g->vdim ? g->dim : g->vdim, f32 ? 4 : 2) + 15) / 16 * 16;
    const int warps = 4 * one <= 200 * 1024 ? 4 : 1;
    const size_t smem = warps * one;
    if (smem > 200 * 1024) return NCB_ERR_UNSUPPORTED;
    if (((uintptr_t)g->conv.proj | (uintptr_t)g->conv.w) % 16 || g->conv.ldp % 8 || g->conv.width % 8 || g->off_q % 8 || (g->own_kv && (g->off_k | g->off_v) % 8))
        return NCB_ERR_ALIGN;
    const int units = g->heads + (g->own_kv ? 2 * g->kv_heads : 0);
    const dim3 grid((units + warps - 1) / warps, (unsigned)((g->conv.rows + RUN - 1) / RUN));
    return f32 ? launch(k_gqa_rows<float>, grid, 32 * warps, smem, 1, (cudaStream_t)stream, *g)
               : launch(k_gqa_rows<bf16>, grid, 32 * warps, smem, 1, (cudaStream_t)stream, *g);
}

/* 1 if gqa_split in bf16 takes these (padded) sizes with q NULL. */
int gqa_split_fused(int dim, int vdim) { return dim > 0 && vdim > 0 && dim <= 256 && vdim <= 256; }

int gqa_split(const ncb_gqa *g, int f32, void *stream) {
    if (!g) return NCB_ERR_ARG;
    int rc = check(*g);
    if (rc != NCB_OK || g->conv.rows == 0) return rc;
    if ((rc = check_parts(*g)) != NCB_OK) return rc;
    if (!f32 && gqa_split_fused(g->dim, g->vdim)) {
        int stages = 4;
        while (stages > 2 && split_smem(g->dim, g->vdim, stages).total > 112 * 1024) stages--;
        const size_t smem = split_smem(g->dim, g->vdim, stages).total;
        const dim3 grid(g->max_chunks, g->kv_heads * ((g->heads / g->kv_heads + HEADS_M - 1) / HEADS_M), (unsigned)g->conv.rows);
        const cudaStream_t s = (cudaStream_t)stream;
        if (g->dim <= 64 && g->vdim <= 64) return launch(k_gqa_split<4, 4>, grid, THREADS, smem, 1, s, *g, stages);
        if (g->dim <= 128 && g->vdim <= 128) return launch(k_gqa_split<8, 8>, grid, THREADS, smem, 1, s, *g, stages);
        return launch(k_gqa_split<16, 16>, grid, THREADS, smem, 1, s, *g, stages);
    }
    if (!g->q) return NCB_ERR_ARG; /* only the form above prepares its rows */
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

int gqa_prefill_supported(int dim, int vdim) { return dim > 0 && vdim > 0 && dim <= 192 && vdim <= 128; }

int gqa_prefill(const ncb_gqa *g, void *stream) {
    if (!g) return NCB_ERR_ARG;
    const int rc = check(*g);
    if (rc != NCB_OK || g->conv.rows == 0 || g->n_tiles == 0) return rc;
    if (!gqa_prefill_supported(g->dim, g->vdim)) return NCB_ERR_UNSUPPORTED;
    if (!g->q || !g->out || g->ldo < g->heads * g->vdim || !g->tile_row || !g->tile_rows || !g->tile_pos || g->n_tiles < 0 || g->n_tiles > 65535)
        return NCB_ERR_ARG;
    const dim3 grid(g->heads, g->n_tiles);
    const size_t smem = (size_t)2 * PF_KEYS * ((g->dim + g->vdim) * 2 + 16);
    const cudaStream_t s = (cudaStream_t)stream;
    if (g->dim == 128 && g->vdim == 128) return launch(k_gqa_prefill<8, 8, true>, grid, THREADS, smem, 1, s, *g);
    if (g->dim == 64 && g->vdim == 64) return launch(k_gqa_prefill<4, 4, true>, grid, THREADS, smem, 1, s, *g);
    return g->dim <= 128 ? launch(k_gqa_prefill<8, 8, false>, grid, THREADS, smem, 1, s, *g)
                         : launch(k_gqa_prefill<12, 8, false>, grid, THREADS, smem, 1, s, *g);
}

} /* extern "C" */
