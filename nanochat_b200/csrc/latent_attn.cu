/*
 * Latent attention: keys and values of all heads are linear images of one cached latent row per position,
 *     k_h = [W_uk,h c | k_rot],  v_h = W_uv,h c,  score = (q_plain . W_uk,h c + q_rot . k_rot) scale,
 * so the cache holds only c (RMS-normed, `rank` values) and the rotated key part k_rot (`rot` values) shared by the heads.
 * Softmax optionally with a sink (exp(sink_h) in the denominator), output optionally gated by sigmoid(gate).
 *
 * Cache: T [n_slots][capacity][rank + rot], T = bf16 (float for a model that runs in 32-bit): a row per position, so all
 * slots are one matrix that TMA reads in boxes, and both contractions read the same bytes.
 *
 * Absorbed form (decode, short portions of prompts): q is taken into latent space, q_abs = [W_uk,h^T q_plain | q_rot],
 * and every head attends the latent rows themselves, as the query heads of ONE key/value head:
 *   - k_latent_query: norm + rotate + append of the new row, rotation of q, and the per-head product with W_uk^T;
 *   - k_latent_split: split over positions. mma.sync m16n8k16 with 16 heads as M; a 32-position tile comes as TMA boxes of 32
 *     rows x 64 columns (128-byte swizzle, conflict-free ldmatrix). Two warps halve the score contraction's depth so that q stays in
 *     registers, two halve the positions; for the second contraction the four warps own a quarter of the latent's columns
 *     each. Scores and probabilities are fp32; a probability enters the second product as two bf16 terms (hi + lo), so its
 *     weight keeps 16 bits. Per (row, head, chunk) an un-normalised state (m in log2 units, l, o);
 *   - k_latent_out: merge of the states, sink, the per-head product with W_uv, gate.
 * Expanded form (prompts): k_latent_append, k_latent_gather (the sequences' latent rows as a matrix, whose product with
 * [W_uk; W_uv] is an ordinary GEMM) and k_latent_prefill: a tile of a prompt's rows against the expanded keys and values.
 * k_latent_split_any and k_latent_out_any are the same steps in plain fp32 arithmetic for any sizes and for T = float.
 */
#include "umma.cuh"

#include <cooperative_groups.h>

namespace cg = cooperative_groups;

namespace {

template <typename T> __device__ __forceinline__ float to_f(T v) { return (float)v; }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16_rn(v); }

constexpr float LOG2E = 1.4426950408889634f;
constexpr int THREADS = 128;
constexpr int TILE = NCB_LATENT_TILE;  /* positions per tile of the split kernel */
constexpr int HEADS_M = 16;            /* heads per block = MMA M */
constexpr int STATE_PAD = 4;           /* floats in front of a state's o: m, l, 2 pad */

__device__ __forceinline__ void mma_bf16(float *d, uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0,
                                         uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, "
                 "{%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm4(uint32_t *r, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4_t(uint32_t *r, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ uint32_t smem_addr(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp_async16(uint32_t dst, const void *src, bool on) { /* 16 bytes, zeros when off */
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(on ? 16 : 0) : "memory");
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

/* Tiles of a row's positions and how they are cut: shared by the split kernels and everything that merges their states. */
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
__device__ __forceinline__ int length_of(const ncb_latent &a, int row, int &slot) {
    const int pos = a.pos[row];
    slot = a.slot_map ? a.slot_map[row] : row;
    if (pos < 0) return 0;
    if (pos >= a.capacity || pos >= a.table_len || slot < 0 || slot >= a.n_slots) {
        flag(a.status, NCB_DEV_BAD_POSITION);
        return 0;
    }
    return pos + 1;
}

/* Two neighbouring values as one load and store. */
template <typename T> __device__ __forceinline__ float2 load2(const T *p);
template <> __device__ __forceinline__ float2 load2<float>(const float *p) { return *reinterpret_cast<const float2 *>(p); }
template <> __device__ __forceinline__ float2 load2<bf16>(const bf16 *p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(p)); }
__device__ __forceinline__ void store2(float *p, float x, float y) { *reinterpret_cast<float2 *>(p) = make_float2(x, y); }
__device__ __forceinline__ void store2(bf16 *p, float x, float y) { *reinterpret_cast<__nv_bfloat162 *>(p) = __floats2bfloat162_rn(x, y); }

/* Rotation of pairs i, i + 1 (i even) of one head's or key's rotated part, from `q` to `out` (may be the same). */
template <typename T> __device__ __forceinline__ void rotate_pairs(const ncb_latent &a, const T *q, T *out, int pos, int i) {
    const int half = a.rot / 2;
    const float2 c = *reinterpret_cast<const float2 *>(a.cos + (size_t)pos * half + i), t = *reinterpret_cast<const float2 *>(a.sin + (size_t)pos * half + i);
    const float2 u = load2<T>(q + i), v = load2<T>(q + half + i);
    store2(out + i, u.x * c.x - v.x * t.x, u.y * c.y - v.y * t.y);
    store2(out + half + i, v.x * c.x + u.x * t.x, v.y * c.y + u.y * t.y);
}

/* One warp: norm of the latent, rotation of the key part, one cache row. */
template <typename T> __device__ __forceinline__ void append_row(const ncb_latent &a, int row, int lane) {
    int slot;
    const int len = length_of(a, row, slot);
    if (len == 0) return;
    const T *kv = (const T *)a.proj + (size_t)row * a.ldp + a.off_kv;
    T *out = (T *)a.cache + ((size_t)slot * a.capacity + (len - 1)) * (a.rank + a.rot);
    float s = 0.f;
#pragma unroll 8
    for (int i = lane * 2; i < a.rank; i += 64) {
        const float2 v = load2<T>(kv + i);
        s = fmaf(v.x, v.x, fmaf(v.y, v.y, s));
    }
    for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    const float rstd = 1.f / sqrtf(s / (float)a.norm_count + a.eps);
#pragma unroll 8
    for (int i = lane * 2; i < a.rank; i += 64) {
        const float2 v = load2<T>(kv + i), w = *reinterpret_cast<const float2 *>(a.norm + i);
        store2(out + i, v.x * rstd * w.x, v.y * rstd * w.y);
    }
    for (int i = lane * 2; i < a.rot / 2; i += 64) rotate_pairs(a, kv + a.rank, out + a.rank, len - 1, i);
}

/* ---- absorbed form: query ------------------------------------------------------------------------------------------- */

/* Grid (rank / 64 rounded up, + 1, heads, ceil(rows / 16)). Block x < last: 64 latent columns of q_abs for one head and 16
 * rows, its weights on their way to shared memory before the dependency wait; block x == last: the rotated part of that
 * head's q, and the appends of the rows dealt to that head. */
template <typename T> __global__ void __launch_bounds__(THREADS) k_latent_query(const ncb_latent a) {
    extern __shared__ __align__(128) uint8_t raw[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y, r0 = blockIdx.z * 16;
    const int W = a.rank + a.rot, stride_q = a.dim + a.rot, f0 = blockIdx.x * 64, ws = a.dim + 8;
    const bool rotate = blockIdx.x == gridDim.x - 1;
    if (sizeof(T) == 2 && !rotate) {
        const int n = min(64, a.rank - f0), per = a.dim / 8;
        const bf16 *src = (const bf16 *)a.w_uk_t + ((size_t)h * a.rank + f0) * a.dim;
        for (int i = tid; i < n * per; i += THREADS) cp_async16(smem_addr(raw) + (i / per * ws + i % per * 8) * 2, src + (size_t)i * 8, true);
        asm volatile("cp.async.commit_group;" ::: "memory");
    }
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const int rows = (int)(a.rows - r0 < 16 ? a.rows - r0 : 16);
    const T *q = (const T *)a.proj + a.off_q + (size_t)h * stride_q;
    T *out = (T *)a.q_abs;
    if (rotate) {
        for (int r = h + warp * a.heads; r < rows; r += a.heads * (THREADS / 32)) append_row<T>(a, r0 + r, lane);
        const int pairs = a.rot / 4;
        for (int i = tid; i < rows * pairs; i += THREADS) {
            const int row = r0 + i / pairs, pos = a.pos[row];
            if (pos >= 0 && pos < a.table_len)
                rotate_pairs(a, q + (size_t)row * a.ldp + a.dim, out + ((size_t)row * a.heads + h) * W + a.rank, pos, i % pairs * 2);
        }
        return;
    }
    if constexpr (sizeof(T) == 2) {
        /* 16 rows x 16 columns per warp, depth dim: the same permutation of the k slots for both operands, 32 k-values per
         * 16-byte load */
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        const int g = lane >> 2, t = lane & 3, c0 = f0 + warp * 16;
        if (c0 >= a.rank) return;
        const bf16 *ws0 = reinterpret_cast<const bf16 *>(raw) + warp * 16 * ws;
        float acc[2][2][4] = {};
        const T *xl = q + (size_t)(r0 + g) * a.ldp + 8 * t, *xh = xl + (size_t)8 * a.ldp;
        const bool lo_on = g < rows, hi_on = g + 8 < rows;
#pragma unroll 4
        for (int k = 0; k < a.dim; k += 32) {
            const uint4 z = make_uint4(0u, 0u, 0u, 0u);
            const uint4 lo = lo_on ? *reinterpret_cast<const uint4 *>(xl + k) : z, hi = hi_on ? *reinterpret_cast<const uint4 *>(xh + k) : z;
#pragma unroll
            for (int j = 0; j < 2; j++) {
                const uint4 b = *reinterpret_cast<const uint4 *>(ws0 + (j * 8 + g) * ws + k + 8 * t);
                mma_bf16(acc[j][0], lo.x, hi.x, lo.y, hi.y, b.x, b.y);
                mma_bf16(acc[j][1], lo.z, hi.z, lo.w, hi.w, b.z, b.w);
            }
        }
#pragma unroll
        for (int j = 0; j < 2; j++)
#pragma unroll
            for (int r = 0; r < 2; r++)
                if (g + 8 * r < rows)
                    *reinterpret_cast<uint32_t *>(out + ((size_t)(r0 + g + 8 * r) * a.heads + h) * W + c0 + j * 8 + 2 * t) =
                        pack_bf16(acc[j][0][2 * r] + acc[j][1][2 * r], acc[j][0][2 * r + 1] + acc[j][1][2 * r + 1]);
    } else {
        const T *w = (const T *)a.w_uk_t + (size_t)h * a.rank * a.dim; /* [rank][dim] of this head */
        const int cols = a.rank - f0 < 64 ? a.rank - f0 : 64;
        for (int i = tid; i < rows * cols; i += THREADS) {
            const int row = r0 + i / cols, c = f0 + i % cols;
            const T *x = q + (size_t)row * a.ldp, *y = w + (size_t)c * a.dim;
            float s = 0.f;
            for (int k = 0; k < a.dim; k++) s = fmaf(to_f(x[k]), to_f(y[k]), s);
            out[((size_t)row * a.heads + h) * W + c] = from_f<T>(s);
        }
    }
}

/* ---- absorbed form: split over positions ---------------------------------------------------------------------------- */

constexpr int BOX_BYTES = TILE * 128; /* 32 rows of 64 bf16 columns */

template <int STAGES> struct SplitSmem {
    __host__ __device__ static int boxes(int W) { return (W + 63) / 64; }
    __host__ __device__ static int bytes(int W) { return 1024 + STAGES * boxes(W) * BOX_BYTES + 2 * HEADS_M * (TILE + 4) * 4 + 64; }
};

/* Grid (max chunks, ceil(heads / 16), rows). MK: 16-wide k-steps per half of the score contraction; MN: 16-wide column
 * tiles of the latent per warp. map: all slots' rows as one matrix [n_slots capacity][rank + rot], boxes of 32 x 64. */
template <int MK, int MN, int STAGES>
__global__ void __launch_bounds__(THREADS, 2) k_latent_split(const __grid_constant__ CUtensorMap map, const ncb_latent a) {
    extern __shared__ __align__(128) uint8_t raw[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int W = a.rank + a.rot, boxes = SplitSmem<STAGES>::boxes(W), stage_bytes = boxes * BOX_BYTES;
    const uint32_t ring = (smem_addr(raw) + 1023u) & ~1023u; /* swizzled boxes sit on 1024-byte boundaries */
    uint8_t *ring_ptr = raw + (ring - smem_addr(raw));
    float *scores = reinterpret_cast<float *>(ring_ptr + STAGES * stage_bytes); /* [2][16][TILE + 4]: the two depth halves */
    const uint32_t bars = ring + STAGES * stage_bytes + 2 * HEADS_M * (TILE + 4) * 4;
    if (tid == 0) {
        for (int s = 0; s < STAGES; s++) mbar_init(bars + 8 * s, 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
        asm volatile("prefetch.tensormap [%0];" ::"l"(&map) : "memory");
    }
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const int row = blockIdx.z, h0 = blockIdx.y * HEADS_M;
    int slot;
    const Cut cut = cut_of(length_of(a, row, slot), a.chunk_tiles);
    const int t0 = blockIdx.x * cut.per, t1 = min(t0 + cut.per, cut.tiles);
    if (blockIdx.x >= cut.n_chunks || t0 >= t1) return;
    __syncthreads();
    const uint64_t policy = policy_evict_first();
    auto fetch = [&](int i) { /* one thread: a tile's boxes */
        const int s = i % STAGES, r = slot * a.capacity + (t0 + i) * TILE;
        mbar_expect_tx(bars + 8 * s, stage_bytes);
        for (int b = 0; b < boxes; b++) tma_load(ring + s * stage_bytes + b * BOX_BYTES, &map, b * 64, r, bars + 8 * s, policy);
    };
    /* the address of 16-byte chunk c of row r in a stage */
    auto chunk_at = [](uint32_t stage, int r, int c) { return stage + (c >> 3) * BOX_BYTES + r * 128 + (((c & 7) ^ (r & 7)) << 4); };
    const int n_tiles = t1 - t0;
    if (tid == 0)
        for (int i = 0; i < min(STAGES, n_tiles); i++) fetch(i);

    /* this warp's half of the score depth, as A operand fragments */
    const int ph = warp & 1, kh = warp >> 1, steps = W / 16, k_half = (steps + 1) / 2;
    const int ks0 = kh * k_half, nks = kh == 0 ? k_half : steps - k_half;
    uint32_t qf[MK][4];
    {
        const bf16 *q = (const bf16 *)a.q_abs + ((size_t)row * a.heads + h0) * W + 2 * t;
        const bool lo_on = h0 + g < a.heads, hi_on = h0 + g + 8 < a.heads;
#pragma unroll
        for (int i = 0; i < MK; i++) {
            const bf16 *p = q + (size_t)g * W + (ks0 + i) * 16;
            const bool on = i < nks;
            qf[i][0] = on && lo_on ? *reinterpret_cast<const uint32_t *>(p) : 0u;
            qf[i][1] = on && hi_on ? *reinterpret_cast<const uint32_t *>(p + (size_t)8 * W) : 0u;
            qf[i][2] = on && lo_on ? *reinterpret_cast<const uint32_t *>(p + 8) : 0u;
            qf[i][3] = on && hi_on ? *reinterpret_cast<const uint32_t *>(p + (size_t)8 * W + 8) : 0u;
        }
    }
    const int col_tiles = a.rank / 16, per_warp = (col_tiles + 3) / 4, ct0 = warp * per_warp;
    const int nct = max(0, min(per_warp, col_tiles - ct0));
    float o[MN][2][4];
#pragma unroll
    for (int i = 0; i < MN; i++)
#pragma unroll
        for (int j = 0; j < 8; j++) o[i][j >> 2][j & 3] = 0.f;
    float m_lo = -INFINITY, m_hi = -INFINITY, l_lo = 0.f, l_hi = 0.f;
    const float scale = a.scale * LOG2E;
    bool ok = true;
    for (int i = 0; i < n_tiles; i++) {
        const int s = i % STAGES, p0 = (t0 + i) * TILE;
        const uint32_t stage = ring + s * stage_bytes;
        if (!mbar_wait(bars + 8 * s, (i / STAGES) & 1)) ok = false;
        __syncwarp();
        const int live = min(TILE, cut.len - p0);
        if (live < TILE) { /* the sequence's last tile: whatever lies past its end must not reach the second product */
            for (int j = tid; j < (TILE - live) * boxes * 8; j += THREADS)
                *reinterpret_cast<uint4 *>(ring_ptr + s * stage_bytes + (j >> 3) / (TILE - live) * BOX_BYTES + (live + (j >> 3) % (TILE - live)) * 128 +
                                           (j & 7) * 16) = make_uint4(0u, 0u, 0u, 0u);
            __syncthreads();
        }
        { /* scores of 16 positions over half of the depth */
            float acc[2][2][4] = {};
            const int r = ph * 16 + (lane >> 4) * 8 + (lane & 7), c = 2 * ks0 + ((lane >> 3) & 1);
#pragma unroll
            for (int ks = 0; ks < MK; ks++)
                if (ks < nks) {
                    uint32_t b[4];
                    ldsm4(b, chunk_at(stage, r, c + 2 * ks));
                    mma_bf16(acc[ks & 1][0], qf[ks][0], qf[ks][1], qf[ks][2], qf[ks][3], b[0], b[1]);
                    mma_bf16(acc[ks & 1][1], qf[ks][0], qf[ks][1], qf[ks][2], qf[ks][3], b[2], b[3]);
                }
            float *sp = scores + kh * HEADS_M * (TILE + 4) + ph * 16 + 2 * t;
#pragma unroll
            for (int n = 0; n < 2; n++) {
                *reinterpret_cast<float2 *>(sp + g * (TILE + 4) + n * 8) = make_float2(acc[0][n][0] + acc[1][n][0], acc[0][n][1] + acc[1][n][1]);
                *reinterpret_cast<float2 *>(sp + (g + 8) * (TILE + 4) + n * 8) = make_float2(acc[0][n][2] + acc[1][n][2], acc[0][n][3] + acc[1][n][3]);
            }
        }
        __syncthreads();
        /* every warp: all 16 x 32 probabilities in A operand layout */
        float p[2][8]; /* [16-position step][lo 0, 1, hi 0, 1, lo 8, 9, hi 8, 9] */
        float mx_lo = m_lo, mx_hi = m_hi;
#pragma unroll
        for (int j = 0; j < 2; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int head = g + (e & 1) * 8, col = j * 16 + 2 * t + (e >> 1) * 8;
                const float2 x = *reinterpret_cast<const float2 *>(scores + head * (TILE + 4) + col);
                const float2 y = *reinterpret_cast<const float2 *>(scores + (HEADS_M + head) * (TILE + 4) + col);
                const float s0 = col < live ? (x.x + y.x) * scale : -INFINITY, s1 = col + 1 < live ? (x.y + y.y) * scale : -INFINITY;
                p[j][2 * e] = s0, p[j][2 * e + 1] = s1;
                if (e & 1) mx_hi = fmaxf(mx_hi, fmaxf(s0, s1));
                else mx_lo = fmaxf(mx_lo, fmaxf(s0, s1));
            }
        mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 1));
        mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 2));
        mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 1));
        mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 2));
        const bool moved = mx_lo != m_lo || mx_hi != m_hi;
        if (__any_sync(0xffffffffu, moved)) {
            const float al = ex2(m_lo - mx_lo), ah = ex2(m_hi - mx_hi); /* 0 for the first tile */
            l_lo *= al, l_hi *= ah;
#pragma unroll
            for (int c = 0; c < MN; c++)
#pragma unroll
                for (int n = 0; n < 2; n++) o[c][n][0] *= al, o[c][n][1] *= al, o[c][n][2] *= ah, o[c][n][3] *= ah;
            m_lo = mx_lo, m_hi = mx_hi;
        }
        uint32_t hi[2][4], lo[2][4];
#pragma unroll
        for (int j = 0; j < 2; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const float m = (e & 1) ? m_hi : m_lo;
                const float a0 = ex2(p[j][2 * e] - m), a1 = ex2(p[j][2 * e + 1] - m);
                if (e & 1) l_hi += a0 + a1;
                else l_lo += a0 + a1;
                split_bf16(a0, a1, hi[j][e], lo[j][e]);
            }
#pragma unroll
        for (int c = 0; c < MN; c++)
            if (c < nct) {
#pragma unroll
                for (int j = 0; j < 2; j++) {
                    uint32_t b[4];
                    ldsm4_t(b, chunk_at(stage, j * 16 + (lane & 15), 2 * (ct0 + c) + (lane >> 4)));
                    mma_bf16(o[c][0], hi[j][0], hi[j][1], hi[j][2], hi[j][3], b[0], b[1]);
                    mma_bf16(o[c][1], hi[j][0], hi[j][1], hi[j][2], hi[j][3], b[2], b[3]);
                    mma_bf16(o[c][0], lo[j][0], lo[j][1], lo[j][2], lo[j][3], b[0], b[1]);
                    mma_bf16(o[c][1], lo[j][0], lo[j][1], lo[j][2], lo[j][3], b[2], b[3]);
                }
            }
        __syncthreads(); /* the stage and the scores may be overwritten */
        if (tid == 0 && i + STAGES < n_tiles) fetch(i + STAGES);
    }
    if (!ok && lane == 0) flag(a.status, NCB_DEV_WAIT_TIMEOUT);
    l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 1);
    l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 2);
    l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 1);
    l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 2);
    const size_t state = (size_t)(a.rank + STATE_PAD);
    float *lo_out = a.parts + (((size_t)row * a.heads + h0 + g) * gridDim.x + blockIdx.x) * state;
    float *hi_out = lo_out + (size_t)8 * gridDim.x * state;
    const bool lo_on = h0 + g < a.heads, hi_on = h0 + g + 8 < a.heads;
    if (warp == 0 && t == 0) {
        if (lo_on) *reinterpret_cast<float2 *>(lo_out) = make_float2(m_lo, l_lo);
        if (hi_on) *reinterpret_cast<float2 *>(hi_out) = make_float2(m_hi, l_hi);
    }
#pragma unroll
    for (int c = 0; c < MN; c++)
        if (c < nct)
#pragma unroll
            for (int n = 0; n < 2; n++) {
                const int col = STATE_PAD + (ct0 + c) * 16 + n * 8 + 2 * t;
                if (lo_on) *reinterpret_cast<float2 *>(lo_out + col) = make_float2(o[c][n][0], o[c][n][1]);
                if (hi_on) *reinterpret_cast<float2 *>(hi_out + col) = make_float2(o[c][n][2], o[c][n][3]);
            }
}

/* The same states in plain fp32 arithmetic: grid (max chunks, heads, rows), any rank and rotated size. */
constexpr int ANY_TILE = 128;
template <typename T> __global__ void __launch_bounds__(THREADS) k_latent_split_any(const ncb_latent a) {
    extern __shared__ float sm[]; /* q [rank + rot], o [rank], probabilities [ANY_TILE], reduction [8] */
    const int tid = threadIdx.x, row = blockIdx.z, h = blockIdx.y, W = a.rank + a.rot;
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    int slot;
    const Cut cut = cut_of(length_of(a, row, slot), a.chunk_tiles);
    const int p0 = min(blockIdx.x * cut.per, cut.tiles) * TILE, p1 = min(min((int)(blockIdx.x + 1) * cut.per, cut.tiles) * TILE, cut.len);
    if (blockIdx.x >= cut.n_chunks || p0 >= p1) return;
    float *q = sm, *o = q + W, *p = o + a.rank, *red = p + ANY_TILE;
    const T *qr = (const T *)a.q_abs + ((size_t)row * a.heads + h) * W;
    for (int i = tid; i < W; i += THREADS) q[i] = to_f(qr[i]);
    for (int i = tid; i < a.rank; i += THREADS) o[i] = 0.f;
    __syncthreads();
    const T *cache = (const T *)a.cache + (size_t)slot * a.capacity * W;
    float m = -INFINITY, l = 0.f;
    for (int at = p0; at < p1; at += ANY_TILE) {
        const int n = min(ANY_TILE, p1 - at);
        float s = -INFINITY;
        if (tid < n) {
            const T *c = cache + (size_t)(at + tid) * W;
            float v = 0.f;
            for (int i = 0; i < W; i++) v = fmaf(q[i], to_f(c[i]), v);
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
        for (int i = tid; i < a.rank; i += THREADS) {
            float v = o[i] * shrink;
            for (int j = 0; j < n; j++) v = fmaf(p[j], to_f(cache[(size_t)(at + j) * W + i]), v);
            o[i] = v;
        }
        __syncthreads();
    }
    float *out = a.parts + (((size_t)row * a.heads + h) * gridDim.x + blockIdx.x) * (a.rank + STATE_PAD);
    if (tid == 0) out[0] = m, out[1] = l;
    for (int i = tid; i < a.rank; i += THREADS) out[STATE_PAD + i] = o[i];
}

/* ---- absorbed form: merge, W_uv, gate ------------------------------------------------------------------------------- */

/* The factor of chunk c's state in the merged output of (row, head): 2^(m_c - M) / L with the sink in M and L. One warp. */
__device__ __forceinline__ void merge_weights(const ncb_latent &a, int row, int h, int n_chunks, float *w, int lane) {
    const size_t state = (size_t)(a.rank + STATE_PAD);
    const float *p = a.parts + ((size_t)row * a.heads + h) * a.max_chunks * state;
    float M = a.sink ? a.sink[h] * LOG2E : -INFINITY;
    const float sink = M;
    for (int c = lane; c < n_chunks; c += 32) M = fmaxf(M, p[c * state]);
    for (int o = 16; o > 0; o >>= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, o));
    float L = 0.f;
    for (int c = lane; c < n_chunks; c += 32) {
        const float e = exp2f(p[c * state] - M);
        w[c] = e;
        L = fmaf(e, p[c * state + 1], L);
    }
    for (int o = 16; o > 0; o >>= 1) L += __shfl_xor_sync(0xffffffffu, L, o);
    if (a.sink) L += exp2f(sink - M);
    const float inv = n_chunks > 0 ? 1.f / L : 0.f;
    for (int c = lane; c < n_chunks; c += 32) w[c] *= inv;
}
template <typename T> __device__ __forceinline__ float gate_of(const ncb_latent &a, int row, int at) {
    return a.gated ? 1.f / (1.f + expf(-to_f(((const T *)a.proj)[(size_t)row * a.ldp + a.off_g + at]))) : 1.f;
}

/* Grid (heads, rows), any sizes: merged latent in shared memory, one warp per output value. */
template <typename T> __global__ void __launch_bounds__(THREADS) k_latent_out_any(const ncb_latent a) {
    extern __shared__ float sm[]; /* weights [max_chunks], merged [rank] */
    const int tid = threadIdx.x, lane = tid & 31, h = blockIdx.x, row = blockIdx.y;
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    int slot;
    const int n = cut_of(length_of(a, row, slot), a.chunk_tiles).n_chunks;
    float *w = sm, *o = sm + a.max_chunks;
    const size_t state = (size_t)(a.rank + STATE_PAD);
    const float *p = a.parts + ((size_t)row * a.heads + h) * a.max_chunks * state + STATE_PAD;
    if (tid < 32) merge_weights(a, row, h, n, w, lane);
    __syncthreads();
    for (int i = tid; i < a.rank; i += THREADS) {
        float v = 0.f;
        for (int c = 0; c < n; c++) v = fmaf(w[c], p[c * state + i], v);
        o[i] = v;
    }
    __syncthreads();
    for (int j = tid >> 5; j < a.vdim; j += THREADS / 32) {
        const T *u = (const T *)a.w_uv + ((size_t)h * a.vdim + j) * a.rank;
        float v = 0.f;
        for (int i = lane; i < a.rank; i += 32) v = fmaf(o[i], to_f(u[i]), v);
        for (int s = 16; s > 0; s >>= 1) v += __shfl_xor_sync(0xffffffffu, v, s);
        if (lane == 0) ((T *)a.out)[(size_t)row * a.ldo + h * a.vdim + j] = from_f<T>(v * gate_of<T>(a, row, h * a.vdim + j));
    }
}

constexpr int OUT_THREADS = 256;

/* Grid (slices, heads, ceil(rows / 16)), cluster (slices, 1, 1): a block merges rank / slices latent columns of 16 rows,
 * multiplies them by its columns of W_uv (on their way to shared memory before the dependency wait) for all of the head's
 * values, and the cluster adds the partial products up. */
__global__ void __launch_bounds__(OUT_THREADS) k_latent_out(const ncb_latent a) {
    extern __shared__ __align__(128) uint8_t raw[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int slices = gridDim.x, rank_block = blockIdx.x, h = blockIdx.y, r0 = blockIdx.z * 16;
    const int cols = a.rank / slices, c0 = rank_block * cols, xs = cols + 8, V = a.vdim;
    float *w = reinterpret_cast<float *>(raw);                          /* [16][max_chunks] */
    float *sum = w + 16 * a.max_chunks;                                 /* [16][vdim + 4] partial products */
    bf16 *x = reinterpret_cast<bf16 *>(sum + 16 * (V + 4));             /* [16][cols + 8] merged latent */
    bf16 *u = x + 16 * xs;                                              /* [vdim][cols + 8] */
    __shared__ int n_chunks[16];
    {
        const int per = cols / 8;
        const bf16 *src = (const bf16 *)a.w_uv + (size_t)h * V * a.rank + c0;
        for (int i = tid; i < V * per; i += OUT_THREADS) cp_async16(smem_addr(u + i / per * xs + i % per * 8), src + (size_t)(i / per) * a.rank + i % per * 8, true);
        asm volatile("cp.async.commit_group;" ::: "memory");
    }
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const int rows = (int)(a.rows - r0 < 16 ? a.rows - r0 : 16);
    const size_t state = (size_t)(a.rank + STATE_PAD);
    { /* the factor of every chunk's state, 16 threads per row: 2^(m - M) / L with the sink in M and L */
        const int r = tid >> 4, j = tid & 15;
        int n = 0, slot;
        if (r < rows) n = cut_of(length_of(a, r0 + r, slot), a.chunk_tiles).n_chunks;
        const float *p = a.parts + ((size_t)(r0 + r) * a.heads + h) * a.max_chunks * state;
        const float sink = a.sink ? a.sink[h] * LOG2E : -INFINITY;
        float M = sink, L = 0.f;
        for (int c = j; c < n; c += 16) M = fmaxf(M, p[c * state]);
        for (int o = 8; o > 0; o >>= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, o));
        for (int c = j; c < n; c += 16) {
            const float2 ml = *reinterpret_cast<const float2 *>(p + c * state);
            const float e = exp2f(ml.x - M);
            w[r * a.max_chunks + c] = e;
            L = fmaf(e, ml.y, L);
        }
        for (int o = 8; o > 0; o >>= 1) L += __shfl_xor_sync(0xffffffffu, L, o);
        if (a.sink) L += exp2f(sink - M);
        const float inv = n > 0 ? 1.f / L : 0.f;
        for (int c = j; c < n; c += 16) w[r * a.max_chunks + c] *= inv;
        if (j == 0) n_chunks[r] = n;
    }
    __syncthreads();
    for (int i = tid; i < 16 * (cols / 4); i += OUT_THREADS) {
        const int r = i / (cols / 4), c4 = i % (cols / 4) * 4;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        const int n = n_chunks[r];
        const float *p = a.parts + ((size_t)(r0 + r) * a.heads + h) * a.max_chunks * state + STATE_PAD + c0 + c4;
        const float *f = w + r * a.max_chunks;
        constexpr int AHEAD = 8; /* states whose loads are in flight together */
        for (int c = 0; c < n; c += AHEAD) {
            float4 s[AHEAD];
#pragma unroll
            for (int j = 0; j < AHEAD; j++)
                s[j] = c + j < n ? *reinterpret_cast<const float4 *>(p + (c + j) * state) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int j = 0; j < AHEAD; j++) {
                const float e = c + j < n ? f[c + j] : 0.f;
                v.x = fmaf(e, s[j].x, v.x), v.y = fmaf(e, s[j].y, v.y), v.z = fmaf(e, s[j].z, v.z), v.w = fmaf(e, s[j].w, v.w);
            }
        }
        *reinterpret_cast<uint2 *>(x + r * xs + c4) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    for (int n0 = warp * 8; n0 < V; n0 += OUT_THREADS / 4) { /* 8 output values at a time */
        float acc[2][4] = {};
        const bf16 *wr = u + (n0 + g) * xs + 8 * t, *xl = x + g * xs + 8 * t, *xh = xl + 8 * xs;
#pragma unroll 4
        for (int k = 0; k < cols; k += 32) {
            const uint4 lo = *reinterpret_cast<const uint4 *>(xl + k), hi = *reinterpret_cast<const uint4 *>(xh + k);
            const uint4 b = *reinterpret_cast<const uint4 *>(wr + k);
            mma_bf16(acc[0], lo.x, hi.x, lo.y, hi.y, b.x, b.y);
            mma_bf16(acc[1], lo.z, hi.z, lo.w, hi.w, b.z, b.w);
        }
        float *s = sum + n0 + 2 * t;
        *reinterpret_cast<float2 *>(s + g * (V + 4)) = make_float2(acc[0][0] + acc[1][0], acc[0][1] + acc[1][1]);
        *reinterpret_cast<float2 *>(s + (g + 8) * (V + 4)) = make_float2(acc[0][2] + acc[1][2], acc[0][3] + acc[1][3]);
    }
    cg::cluster_group cluster = cg::this_cluster();
    if (slices > 1) cluster.sync();
    else __syncthreads();
    for (int i = rank_block * OUT_THREADS + tid; i < rows * V; i += slices * OUT_THREADS) {
        const int r = i / V, j = i % V;
        const float gate = gate_of<bf16>(a, r0 + r, h * V + j);
        float v = 0.f;
        for (int s = 0; s < slices; s++) v += slices > 1 ? cluster.map_shared_rank(sum, s)[r * (V + 4) + j] : sum[r * (V + 4) + j];
        ((bf16 *)a.out)[(size_t)(r0 + r) * a.ldo + h * V + j] = __float2bfloat16_rn(v * gate);
    }
    if (slices > 1) cluster.sync(); /* nobody leaves while a peer still reads its shared memory */
}

/* ---- expanded form -------------------------------------------------------------------------------------------------- */

/* Grid (ceil(rows / 4)): a warp per row appends its latent row and rotates the row's q in place. */
template <typename T> __global__ void __launch_bounds__(THREADS) k_latent_append(const ncb_latent a) {
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const int row = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (row >= a.rows) return;
    append_row<T>(a, row, lane);
    const int pos = a.pos[row], pairs = a.rot / 4;
    if (!a.rotate_q || pos < 0 || pos >= a.table_len) return;
    T *q = (T *)a.proj + (size_t)row * a.ldp + a.off_q + a.dim;
#pragma unroll 4
    for (int i = lane; i < a.heads * pairs; i += 32) {
        T *p = q + (size_t)(i / pairs) * (a.dim + a.rot);
        rotate_pairs(a, p, p, pos, i % pairs * 2);
    }
}

/* Grid (ceil(longest context / 4), segments): the cached rows of a segment's whole context as matrices, latent part
 * [ctx][ctx_ld] (columns past rank are zeroed: the GEMM over them wants a multiple of 64) and rotated part [ctx][rot]. */
__global__ void __launch_bounds__(THREADS) k_latent_gather(const ncb_latent a) {
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const int seg = blockIdx.y, p = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    const int slot = a.ctx_slot[seg], first = a.ctx_first[seg], len = a.ctx_first[seg + 1] - first;
    if (p >= len) return;
    const bool ok = slot >= 0 && slot < a.n_slots && p < a.capacity;
    if (!ok && p == 0 && lane == 0) flag(a.status, NCB_DEV_BAD_POSITION);
    const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
    const uint4 *src = reinterpret_cast<const uint4 *>((const bf16 *)a.cache + ((size_t)(ok ? slot : 0) * a.capacity + (ok ? p : 0)) * (a.rank + a.rot));
    uint4 *c = reinterpret_cast<uint4 *>((bf16 *)a.ctx + (size_t)(first + p) * a.ctx_ld), *k = reinterpret_cast<uint4 *>((bf16 *)a.ctx_rot + (size_t)(first + p) * a.rot);
    for (int i = lane; i < a.ctx_ld / 8; i += 32) c[i] = ok && i < a.rank / 8 ? src[i] : zero;
    for (int i = lane; i < a.rot / 8; i += 32) k[i] = ok ? src[a.rank / 8 + i] : zero;
}

constexpr int PF_ROWS = 64, PF_KEYS = 64; /* query rows and keys per tile: four warps of 16 rows */

/* Grid (heads, row tiles): PF_ROWS consecutive rows of one sequence against its expanded keys and values, one head. Keys
 * and values of 64 positions per stage (cp.async, two stages); a warp owns 16 rows over the whole range: scores, fp32
 * softmax and the second product (probabilities as two bf16 terms) in registers. QS: 16-wide steps of the score depth;
 * VN: 16-wide column tiles of the values (both upper bounds, or with EXACT the sizes). */
template <int QS, int VN, bool EXACT> __global__ void __launch_bounds__(THREADS, 2) k_latent_prefill(const ncb_latent a) {
    extern __shared__ __align__(128) uint8_t raw[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int h = blockIdx.x, tile = blockIdx.y, depth = EXACT ? QS * 16 : a.dim + a.rot, vdim = EXACT ? VN * 16 : a.vdim;
    const int steps = depth / 16, cols = vdim / 16;
    const int krow = depth * 2 + 16, vrow = vdim * 2 + 16, stage_bytes = PF_KEYS * (krow + vrow);
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const int row0 = a.tile_row[tile], n_rows = min(a.tile_rows[tile], PF_ROWS), ctx0 = a.tile_ctx[tile], pos0 = a.tile_pos[tile];
    const int keys = pos0 + n_rows, n_tiles = (keys + PF_KEYS - 1) / PF_KEYS; /* the last row sees positions < keys */
    const uint32_t smem = smem_addr(raw);
    const bf16 *kv = (const bf16 *)a.ctx_kv + (size_t)ctx0 * a.ctx_kv_ld + (size_t)h * (a.dim + a.vdim);
    const bf16 *kr = (const bf16 *)a.ctx_rot + (size_t)ctx0 * a.rot;
    auto fetch = [&](int i) {
        const uint32_t ks = smem + (i & 1) * stage_bytes, vs = ks + PF_KEYS * krow;
        const int p0 = i * PF_KEYS, nd = a.dim / 8, nr = a.rot / 8, nv = a.vdim / 8, c0 = tid & 7;
#pragma unroll
        for (int j = 0; j < PF_KEYS / 16; j++) { /* eight threads per row, 16 rows at a time */
            const int r = (tid >> 3) + 16 * j;
            const bool on = p0 + r < keys;
            const bf16 *src = kv + (size_t)(on ? p0 + r : 0) * a.ctx_kv_ld, *rot = kr + (size_t)(on ? p0 + r : 0) * a.rot;
            const uint32_t kd = ks + r * krow, vd = vs + r * vrow;
            for (int c = c0; c < nd; c += 8) cp_async16(kd + c * 16, src + c * 8, on);
            for (int c = c0; c < nr; c += 8) cp_async16(kd + (nd + c) * 16, rot + c * 8, on);
            for (int c = c0; c < nv; c += 8) cp_async16(vd + c * 16, src + a.dim + c * 8, on);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(0);
    uint32_t qf[QS][4];
    const int lo_row = warp * 16 + g, hi_row = lo_row + 8;
    const bool lo_on = lo_row < n_rows, hi_on = hi_row < n_rows;
    {
        const bf16 *q = (const bf16 *)a.proj + (size_t)row0 * a.ldp + a.off_q + (size_t)h * depth + 2 * t;
        const bf16 *lo = q + (size_t)lo_row * a.ldp, *hi = q + (size_t)hi_row * a.ldp;
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
        const uint32_t ks = smem + (i & 1) * stage_bytes, vs = ks + PF_KEYS * krow;
        const int p0 = i * PF_KEYS;
        if (p0 <= warp_last) { /* some row of this warp sees some key of the tile */
            float s[PF_KEYS / 8][4];
#pragma unroll
            for (int n = 0; n < PF_KEYS / 8; n++) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
            const uint32_t kbase = ks + ((lane >> 4) * 8 + (lane & 7)) * krow + ((lane >> 3) & 1) * 16;
#pragma unroll
            for (int k = 0; k < QS; k++)
                if (k < steps) {
#pragma unroll
                    for (int n = 0; n < PF_KEYS / 16; n++) {
                        uint32_t b[4];
                        ldsm4(b, kbase + n * 16 * krow + k * 32);
                        mma_bf16(s[2 * n], qf[k][0], qf[k][1], qf[k][2], qf[k][3], b[0], b[1]);
                        mma_bf16(s[2 * n + 1], qf[k][0], qf[k][1], qf[k][2], qf[k][3], b[2], b[3]);
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
            const uint32_t vbase = vs + (lane & 15) * vrow + (lane >> 4) * 16;
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
                        ldsm4_t(b, vbase + j * 16 * vrow + c * 32);
                        mma_bf16(o[c][0], hi[0], hi[1], hi[2], hi[3], b[0], b[1]);
                        mma_bf16(o[c][1], hi[0], hi[1], hi[2], hi[3], b[2], b[3]);
                        mma_bf16(o[c][0], lo[0], lo[1], lo[2], lo[3], b[0], b[1]);
                        mma_bf16(o[c][1], lo[0], lo[1], lo[2], lo[3], b[2], b[3]);
                    }
            }
        }
        __syncthreads(); /* the stage may be overwritten */
    }
    l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 1);
    l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 2);
    l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 1);
    l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 2);
    float f_lo = 1.f, f_hi = 1.f;
    if (a.sink) {
        const float sink = a.sink[h] * LOG2E, ml = fmaxf(m_lo, sink), mh = fmaxf(m_hi, sink);
        f_lo = exp2f(m_lo - ml), f_hi = exp2f(m_hi - mh);
        l_lo = fmaf(l_lo, f_lo, exp2f(sink - ml)), l_hi = fmaf(l_hi, f_hi, exp2f(sink - mh));
    }
    f_lo /= l_lo, f_hi /= l_hi;
#pragma unroll
    for (int c = 0; c < VN; c++)
        if (c < cols)
#pragma unroll
            for (int n = 0; n < 2; n++)
#pragma unroll
                for (int r = 0; r < 2; r++)
                    if (r ? hi_on : lo_on) {
                        const int row = row0 + (r ? hi_row : lo_row), at = h * a.vdim + c * 16 + n * 8 + 2 * t;
                        const float f = r ? f_hi : f_lo;
                        float g0 = 1.f, g1 = 1.f;
                        if (a.gated) {
                            const float2 z = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>((const bf16 *)a.proj + (size_t)row * a.ldp + a.off_g + at));
                            g0 = 1.f / (1.f + expf(-z.x)), g1 = 1.f / (1.f + expf(-z.y));
                        }
                        *reinterpret_cast<uint32_t *>((bf16 *)a.out + (size_t)row * a.ldo + at) =
                            pack_bf16(o[c][n][2 * r] * f * g0, o[c][n][2 * r + 1] * f * g1);
                    }
}

/* ---- host side ------------------------------------------------------------------------------------------------------ */

template <typename... A>
int launch(void (*kernel)(A...), dim3 grid, size_t smem, int threads, int cluster, cudaStream_t stream, A... args) {
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

int check(const ncb_latent &g) {
    if (g.rows < 0 || g.rows > 0x7fffff00LL || g.heads <= 0 || g.heads > 65535 || g.dim <= 0 || g.rot <= 0 || g.vdim <= 0 ||
        g.rank <= 0 || g.dim % 32 || g.rot % 16 || g.vdim % 16 || g.rank % 32 || g.norm_count <= 0 || g.norm_count > g.rank ||
        g.n_slots <= 0 || g.capacity <= 0 || g.table_len <= 0)
        return NCB_ERR_ARG;
    if (g.rows == 0) return NCB_OK;
    if (!g.proj || !g.cache || !g.norm || !g.cos || !g.sin || !g.pos) return NCB_ERR_ARG;
    if (g.ldp % 8 || g.off_q % 8 || g.off_kv % 8 || g.off_g % 8) return NCB_ERR_ALIGN;
    return ((uintptr_t)g.proj | (uintptr_t)g.cache | (uintptr_t)g.q_abs | (uintptr_t)g.parts | (uintptr_t)g.w_uk_t | (uintptr_t)g.w_uv) % 16
               ? NCB_ERR_ALIGN : NCB_OK;
}

template <int MK, int MN, int STAGES> int launch_split(const ncb_latent &g, cudaStream_t s) {
    CUtensorMap map;
    if (!tensor_map(g.cache, g.n_slots * g.capacity, g.rank + g.rot, TILE, &map)) return NCB_ERR_LAUNCH;
    return launch(k_latent_split<MK, MN, STAGES>, dim3(g.max_chunks, (g.heads + HEADS_M - 1) / HEADS_M, (unsigned)g.rows),
                  (size_t)SplitSmem<STAGES>::bytes(g.rank + g.rot), THREADS, 1, s, map, g);
}

} /* namespace */

extern "C" {

int latent_append(const ncb_latent *g, int f32, void *stream) {
    if (!g) return NCB_ERR_ARG;
    const int rc = check(*g);
    if (rc != NCB_OK || g->rows == 0) return rc;
    const dim3 grid((unsigned)((g->rows + 3) / 4));
    return f32 ? launch(k_latent_append<float>, grid, 0, THREADS, 1, (cudaStream_t)stream, *g)
               : launch(k_latent_append<bf16>, grid, 0, THREADS, 1, (cudaStream_t)stream, *g);
}

int latent_query(const ncb_latent *g, int f32, void *stream) {
    if (!g) return NCB_ERR_ARG;
    const int rc = check(*g);
    if (rc != NCB_OK || g->rows == 0) return rc;
    if (!g->q_abs || !g->w_uk_t || (g->rows + 15) / 16 > 65535) return NCB_ERR_ARG;
    const dim3 grid((g->rank + 63) / 64 + 1, g->heads, (unsigned)((g->rows + 15) / 16));
    const size_t smem = f32 ? 0 : (size_t)64 * (g->dim + 8) * 2;
    if (smem > 200 * 1024) return NCB_ERR_UNSUPPORTED;
    return f32 ? launch(k_latent_query<float>, grid, smem, THREADS, 1, (cudaStream_t)stream, *g)
               : launch(k_latent_query<bf16>, grid, smem, THREADS, 1, (cudaStream_t)stream, *g);
}

int latent_split(const ncb_latent *g, int f32, void *stream) {
    if (!g) return NCB_ERR_ARG;
    const int rc = check(*g);
    if (rc != NCB_OK || g->rows == 0) return rc;
    if (!g->q_abs || !g->parts || g->chunk_tiles <= 0 || g->max_chunks <= 0 || g->rows > 65535) return NCB_ERR_ARG;
    if ((long long)g->max_chunks * g->chunk_tiles < (g->max_len + TILE - 1) / TILE || g->max_len <= 0) return NCB_ERR_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    const int half = ((g->rank + g->rot) / 16 + 1) / 2, per_warp = (g->rank / 16 + 3) / 4;
    if (!f32 && g->capacity % TILE == 0 && (long long)g->n_slots * g->capacity < 0x7fffffffLL) {
        if (half <= 3 && per_warp <= 1) return launch_split<3, 1, 4>(*g, s);
        if (half <= 6 && per_warp <= 2) return launch_split<6, 2, 4>(*g, s);
        if (half <= 10 && per_warp <= 4) return launch_split<10, 4, 3>(*g, s);
        if (half <= 20 && per_warp <= 8) return launch_split<20, 8, 2>(*g, s);
    }
    const size_t smem = ((size_t)2 * g->rank + g->rot + ANY_TILE + 8) * sizeof(float);
    if (smem > 200 * 1024) return NCB_ERR_UNSUPPORTED;
    const dim3 grid(g->max_chunks, g->heads, (unsigned)g->rows);
    return f32 ? launch(k_latent_split_any<float>, grid, smem, THREADS, 1, s, *g) : launch(k_latent_split_any<bf16>, grid, smem, THREADS, 1, s, *g);
}

int latent_out(const ncb_latent *g, int f32, void *stream) {
    if (!g) return NCB_ERR_ARG;
    const int rc = check(*g);
    if (rc != NCB_OK || g->rows == 0) return rc;
    if (!g->parts || !g->w_uv || !g->out || g->chunk_tiles <= 0 || g->max_chunks <= 0 || g->rows > 65535) return NCB_ERR_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    if (!f32) {
        int slices = 4;
        while (slices > 1 && g->rank % (slices * 32)) slices /= 2;
        const size_t smem = (size_t)16 * g->max_chunks * 4 + (size_t)16 * (g->vdim + 4) * 4 + (size_t)(16 + g->vdim) * (g->rank / slices + 8) * 2;
        if (smem <= 200 * 1024)
            return launch(k_latent_out, dim3(slices, g->heads, (unsigned)((g->rows + 15) / 16)), smem, OUT_THREADS, slices, s, *g);
    }
    const size_t smem = ((size_t)g->max_chunks + g->rank) * sizeof(float);
    if (smem > 200 * 1024) return NCB_ERR_UNSUPPORTED;
    const dim3 grid(g->heads, (unsigned)g->rows);
    return f32 ? launch(k_latent_out_any<float>, grid, smem, THREADS, 1, s, *g) : launch(k_latent_out_any<bf16>, grid, smem, THREADS, 1, s, *g);
}

int latent_gather(const ncb_latent *g, void *stream) {
    if (!g) return NCB_ERR_ARG;
    const int rc = check(*g);
    if (rc != NCB_OK || g->n_contexts == 0) return rc;
    if (!g->ctx || !g->ctx_rot || !g->ctx_slot || !g->ctx_first || g->n_contexts < 0 || g->n_contexts > 65535 || g->max_len <= 0 ||
        g->ctx_ld < g->rank || g->ctx_ld % 8)
        return NCB_ERR_ARG;
    return launch(k_latent_gather, dim3((g->max_len + 3) / 4, g->n_contexts), 0, THREADS, 1, (cudaStream_t)stream, *g);
}

/* 1 if latent_prefill takes these (padded) sizes. */
int latent_prefill_supported(int dim, int rot, int vdim) {
    return dim > 0 && rot > 0 && vdim > 0 && dim % 32 == 0 && rot % 16 == 0 && vdim % 16 == 0 && dim + rot <= 192 && vdim <= 128;
}

int latent_prefill(const ncb_latent *g, void *stream) {
    if (!g) return NCB_ERR_ARG;
    const int rc = check(*g);
    if (rc != NCB_OK || g->n_tiles == 0) return rc;
    if (!latent_prefill_supported(g->dim, g->rot, g->vdim)) return NCB_ERR_UNSUPPORTED;
    if (!g->ctx_kv || !g->ctx_rot || !g->out || !g->tile_row || !g->tile_rows || !g->tile_ctx || !g->tile_pos || g->n_tiles < 0 ||
        g->n_tiles > 65535 || g->ctx_kv_ld < g->heads * (g->dim + g->vdim) || g->ctx_kv_ld % 8 || g->ldo % 2)
        return NCB_ERR_ARG;
    const dim3 grid(g->heads, g->n_tiles);
    const size_t smem = (size_t)2 * PF_KEYS * ((g->dim + g->rot) * 2 + 16 + g->vdim * 2 + 16);
    cudaStream_t s = (cudaStream_t)stream;
    if (g->dim + g->rot == 192 && g->vdim == 128) return launch(k_latent_prefill<12, 8, true>, grid, smem, THREADS, 1, s, *g);
    return g->dim + g->rot <= 128 ? launch(k_latent_prefill<8, 8, false>, grid, smem, THREADS, 1, s, *g)
                                  : launch(k_latent_prefill<12, 8, false>, grid, smem, THREADS, 1, s, *g);
}

} /* extern "C" */
