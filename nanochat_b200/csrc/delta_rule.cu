/*
 * Gated delta rule with a decay per key channel: per sequence and head a matrix state S [dim][vdim] in fp32,
 *     S <- diag(g_t) S,  u_t = beta_t (v_t - S^T k_t),  S <- S + k_t u_t^T,  o_t = S^T q_t,
 * with g = exp(-exp(A_log) softplus(W_a2 a + dt_bias)), beta = sigmoid(b), q and k unit vectors of convolved, silu'd projections
 * (q times q_scale), followed by an RMS norm of o over vdim with a weight and a low-rank sigmoid gate. The state lives in one
 * buffer per layer, fp32 [n_slots][heads][dim][vdim]; position 0 starts from zero whatever the slot held before.
 * Everything from the convolution on is fp32.
 *
 *   - k_delta_step: token by token. A block (or a cluster of blocks that share the norm's sum through distributed shared
 *     memory) owns a slice of vdim of one head and holds its part of the state in registers for all tokens of the segment. The
 *     decayed state meets k and q in one pass, o = S'^T q + (k . q) u, so a token costs one reduction over the key channels.
 *   - chunks of up to 64 tokens (prompts, bf16 projections, dim <= 256). With G_t the product of the decays since the chunk's
 *     start, S_t = G_t S_0 + sum_(s <= t) (G_t / G_s) k_s u_s^T, and the u of a chunk solve a unit lower triangular system:
 *         (I + A) U = beta (V - (G K) S_0),  A[t][s] = beta_t sum_d k_td k_sd G_td / G_sd  (s < t),
 *     so U = U_0 - W S_0 with (I + A) [W | U_0] = beta [G K | V], which needs no state:
 *       k_delta_chunk   (all chunks in parallel) convolutions, unit norms, decays, A, the solve, and B[t][s] = sum_d q k G_t / G_s;
 *       k_delta_scan    (chunk after chunk) U, and the state S <- G_C S + (K G_C / G)^T U; S^T stays in the accumulators of a
 *                       warp, which owns 16 values of the head, and turns into MMA operands in place;
 *       k_delta_out     (all chunks in parallel) O = (Q G) S_0 + B U, norm, gate.
 *     A decay between two tokens is always a product of the decays between them, never a quotient or a difference of long sums,
 *     so none, however strong, overflows or loses the small ones beside it. Products on the tensor cores take their fp32
 *     operands as two bf16 terms each (three MMAs); the low-rank products have bf16 operands to begin with.
 * T is the type of projections and outputs: bf16, or float for a model that runs in 32-bit.
 */
#include "short_conv.cuh"

#include <cooperative_groups.h>

namespace cg = cooperative_groups;

namespace {

__device__ __forceinline__ float sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float silu(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float decay_of(float z, float a_exp) { return expf(-a_exp * softplus(z)); }
constexpr float UNIT_EPS = 1e-6f;

constexpr int STEP_THREADS = 256, STEP_WARPS = STEP_THREADS / 32;

/* Shared memory of k_delta_step in floats; VS: values per block, dgs: groups of key channels, rank: the larger of the two. */
struct StepSmem {
    int q, k, g, v, low, part, u, sums, total;
};
__host__ __device__ inline StepSmem step_smem(int D, int VS, int dgs, int rank_a, int rank_g) {
    StepSmem s;
    int at = 0;
    auto take = [&](int n) { const int r = at; at += (n + 3) / 4 * 4; return r; };
    const int wide = D > VS ? D : VS;
    s.q = take(D), s.k = take(D), s.g = take(D), s.v = take(VS), s.low = take(rank_a + rank_g);
    const int low_part = STEP_THREADS * 2 > wide ? STEP_THREADS * 2 : wide; /* partial low-rank products */
    s.part = take(2 * dgs * VS > low_part ? 2 * dgs * VS : low_part);
    s.u = take(2 * VS); /* u, then o */
    s.sums = take(4 * STEP_WARPS + 8);
    s.total = at;
    return s;
}

/* y[c] = sum_r w[r][c] x[r] for columns [0, n) of w [rank][ldw] (n even), the depth dealt to groups of threads; the partial
 * sums go to part [groups][n]: groups_of(n). */
__device__ __forceinline__ int groups_of(int n) { return n / 2 >= STEP_THREADS ? 1 : STEP_THREADS / (n / 2); }
template <typename T> __device__ __forceinline__ void low_rank(const T *w, int ldw, int rank, int n, const float *x, float *part, int tid) {
    const int pairs = n / 2, groups = groups_of(n);
    for (int i = tid; i < pairs * groups; i += STEP_THREADS) {
        const int c = 2 * (i % pairs), grp = i / pairs;
        float2 y = make_float2(0.f, 0.f);
#pragma unroll 8
        for (int r = grp; r < rank; r += groups) {
            const float2 v = load2<T>(w + (size_t)r * ldw + c);
            y.x = fmaf(v.x, x[r], y.x), y.y = fmaf(v.y, x[r], y.y);
        }
        *reinterpret_cast<float2 *>(part + grp * n + c) = y;
    }
}

/* Grid (slices, heads, segments), cluster (slices, 1, 1); segment z = rows first[z] .. + count[z] - 1 of one slot at ascending
 * positions (first NULL: row z alone). VS values per block (the last slice may hold fewer), NR key channels per thread. */
template <typename T, int NR> __global__ void __launch_bounds__(STEP_THREADS, NR > 16 ? 1 : 2) k_delta_step(const ncb_delta a, int VS) {
    extern __shared__ float sm[];
    __shared__ float block_sum;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y, slices = gridDim.x, rank = blockIdx.x;
    const int D = a.dim, V = a.vdim, v0 = rank * VS, nv = min(VS, V - v0), kh = h / (a.heads / a.kv_heads);
    const int columns = VS / 4, dgs = STEP_THREADS / columns, c = tid % columns, dg = tid / columns;
    const StepSmem L = step_smem(D, VS, dgs, a.rank_a, a.rank_g);
    float *q = sm + L.q, *k = sm + L.k, *g = sm + L.g, *v = sm + L.v, *low = sm + L.low, *part = sm + L.part, *u = sm + L.u, *o = u + VS,
          *sums = sm + L.sums;
    const int first = a.seg_first ? a.seg_first[blockIdx.z] : blockIdx.z, count = a.seg_first ? a.seg_count[blockIdx.z] : 1;
    cg::cluster_group cluster = cg::this_cluster();
    const int pos0 = a.conv.pos[first], slot = a.conv.slot_map ? a.conv.slot_map[first] : first;
    const bool bad = pos0 >= 0 && (slot < 0 || slot >= a.conv.n_slots), mine = dg < dgs && 4 * c < nv;
    float *state = a.state + ((size_t)(bad ? 0 : slot) * a.heads + h) * D * V + v0 + 4 * c;
    /* Positions, slots and this state were last written many launches ago (the launch before this one writes the projection
     * alone), so the state starts towards registers before the dependency wait. */
    float4 s[NR];
#pragma unroll
    for (int i = 0; i < NR; i++) {
        const int d = dg + i * dgs;
        s[i] = pos0 > 0 && !bad && mine && d < D ? *reinterpret_cast<const float4 *>(state + (size_t)d * V) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    if (bad && tid == 0) flag(a.status, NCB_DEV_BAD_POSITION);
    if (pos0 < 0 || bad) { /* an idle row: no state touched, a zero output (every block of the cluster takes this exit) */
        if (a.out)
            for (int i = tid; i < count * nv; i += STEP_THREADS)
                ((T *)a.out)[(size_t)(first + i / nv) * a.ldo + h * V + v0 + i % nv] = from_f<T>(0.f);
        return;
    }
    const T *a2 = (const T *)a.a2 + (size_t)h * a.rank_a * D, *g2 = (const T *)a.g2 + (size_t)h * a.rank_g * V + v0;
    const bool keep_qk = a.keep && rank == 0 && h % (a.heads / a.kv_heads) == 0;
    for (int t = 0; t < count; t++) {
        const int row = first + t;
        const T *p = (const T *)a.conv.proj + (size_t)row * a.conv.ldp;
        const Place at = place_of(a.conv, row);
        for (int i = tid; i < D + nv / 2; i += STEP_THREADS) { /* pairs of channels: q, k, v */
            const int which = 2 * i / D, j = which < 2 ? 2 * i - which * D : 2 * i - 2 * D;
            const int ch = which == 0 ? a.off_q + kh * D + j : which == 1 ? a.off_k + kh * D + j : a.off_v + h * V + v0 + j;
            const float2 y = conv2<T>(a.conv, row, at, ch);
            *reinterpret_cast<float2 *>((which == 0 ? q : which == 1 ? k : v) + j) = make_float2(silu(y.x), silu(y.y));
            if (a.keep && (which >= 2 || keep_qk)) keep2<T>(a.conv, row, at, ch);
        }
        for (int i = tid; i < a.rank_a + a.rank_g; i += STEP_THREADS)
            low[i] = to_f(i < a.rank_a ? p[a.off_a + i] : p[a.off_g + i - a.rank_a]);
        __syncthreads();
        low_rank<T>(a2, D, a.rank_a, D, low, part, tid);
        if (warp < 3) { /* |q|^2, |k|^2, q . k */
            const float *x = warp == 1 ? k : q, *y = warp == 0 ? q : k;
            float w = 0.f;
            for (int d = lane; d < D; d += 32) w = fmaf(x[d], y[d], w);
            for (int off = 16; off > 0; off >>= 1) w += __shfl_xor_sync(0xffffffffu, w, off);
            if (lane == 0) sums[warp] = w;
        }
        __syncthreads();
        const float qr = a.q_scale / sqrtf(sums[0] + UNIT_EPS), kr = 1.f / sqrtf(sums[1] + UNIT_EPS), qk = sums[2] * qr * kr;
        for (int d = tid; d < D; d += STEP_THREADS) {
            float z = a.dt_bias[h * D + d];
            for (int j = 0; j < groups_of(D); j++) z += part[j * D + d];
            g[d] = decay_of(z, a.a_exp[h]);
            q[d] *= qr, k[d] *= kr;
        }
        __syncthreads();
        if (mine) {
            float4 x = make_float4(0.f, 0.f, 0.f, 0.f), y = x; /* S'^T k, S'^T q over this thread's channels */
#pragma unroll
            for (int i = 0; i < NR; i++) {
                const int d = dg + i * dgs;
                if (d >= D) break;
                const float gd = g[d], kd = k[d], qd = q[d];
                s[i].x *= gd, s[i].y *= gd, s[i].z *= gd, s[i].w *= gd;
                x.x = fmaf(kd, s[i].x, x.x), x.y = fmaf(kd, s[i].y, x.y), x.z = fmaf(kd, s[i].z, x.z), x.w = fmaf(kd, s[i].w, x.w);
                y.x = fmaf(qd, s[i].x, y.x), y.y = fmaf(qd, s[i].y, y.y), y.z = fmaf(qd, s[i].z, y.z), y.w = fmaf(qd, s[i].w, y.w);
            }
            *reinterpret_cast<float4 *>(part + dg * VS + 4 * c) = x;
            *reinterpret_cast<float4 *>(part + (dgs + dg) * VS + 4 * c) = y;
        }
        __syncthreads();
        const float beta = sigmoid(to_f(p[a.off_b + h]));
        float sq = 0.f;
        for (int i = tid; i < nv; i += STEP_THREADS) {
            float x = 0.f, y = 0.f;
            for (int j = 0; j < dgs; j++) x += part[j * VS + i], y += part[(dgs + j) * VS + i];
            const float ui = beta * (v[i] - x), oi = fmaf(qk, ui, y);
            u[i] = ui, o[i] = oi;
            sq = fmaf(oi, oi, sq);
        }
        for (int off = 16; off > 0; off >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, off);
        if (lane == 0) sums[8 + warp] = sq;
        __syncthreads();
        if (mine) {
            const float4 w = *reinterpret_cast<const float4 *>(u + 4 * c);
#pragma unroll
            for (int i = 0; i < NR; i++) {
                const int d = dg + i * dgs;
                if (d >= D) break;
                const float kd = k[d];
                s[i].x = fmaf(kd, w.x, s[i].x), s[i].y = fmaf(kd, w.y, s[i].y), s[i].z = fmaf(kd, w.z, s[i].z), s[i].w = fmaf(kd, w.w, s[i].w);
            }
        }
        if (a.out) {
            low_rank<T>(g2, V, a.rank_g, nv, low + a.rank_a, part, tid);
            if (tid == 0) {
                float w = 0.f;
                for (int j = 0; j < STEP_WARPS; j++) w += sums[8 + j];
                block_sum = w;
            }
            float total;
            if (slices > 1) {
                cluster.sync();
                total = 0.f;
                for (int j = 0; j < slices; j++) total += *cluster.map_shared_rank(&block_sum, j);
                cluster.sync(); /* nobody overwrites its sum, or leaves, while a peer still reads it */
            } else {
                __syncthreads();
                total = block_sum;
            }
            const float rstd = 1.f / sqrtf(total / (float)a.norm_count + a.eps);
            for (int i = tid; i < nv; i += STEP_THREADS) {
                float z = 0.f;
                for (int j = 0; j < groups_of(nv); j++) z += part[j * nv + i];
                ((T *)a.out)[(size_t)row * a.ldo + h * V + v0 + i] = from_f<T>(o[i] * rstd * a.norm[v0 + i] * sigmoid(z));
            }
        }
        __syncthreads(); /* the shared arrays are free for the next token */
    }
    if (mine) {
#pragma unroll
        for (int i = 0; i < NR; i++) {
            const int d = dg + i * dgs;
            if (d < D) *reinterpret_cast<float4 *>(state + (size_t)d * V) = s[i];
        }
    }
}

/* ---- chunked form ----------------------------------------------------------------------------------------------------- */

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
__device__ __forceinline__ uint32_t smem_addr(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ uint32_t bits(__nv_bfloat162 v) { return *reinterpret_cast<uint32_t *>(&v); }
/* hi = bf16(v), lo = bf16(v - hi) of two values: 16 bits of mantissa. */
__device__ __forceinline__ void split2(float x, float y, uint32_t &hi, uint32_t &lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const float2 f = __bfloat1622float2(h);
    hi = bits(h);
    lo = bits(__floats2bfloat162_rn(x - f.x, y - f.y));
}
__device__ __forceinline__ void split1(float x, bf16 *hi, bf16 *lo) {
    const bf16 h = __float2bfloat16_rn(x);
    *hi = h;
    *lo = __float2bfloat16_rn(x - to_f(h));
}
/* The two-term pair (hi, lo) times f0, f1 as a new two-term pair. */
__device__ __forceinline__ void rescale2(uint32_t &hi, uint32_t &lo, float f0, float f1) {
    const float2 h = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&hi)), l = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&lo));
    split2((h.x + l.x) * f0, (h.y + l.y) * f1, hi, lo);
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void *src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
/* v[0 .. 63] summed over the warp by halving: lane l ends up with the sums of values 2 l and 2 l + 1 in v[0], v[1]. */
__device__ __forceinline__ void reduce64(float (&v)[64], int lane) {
#pragma unroll
    for (int step = 0; step < 5; step++) {
        const int n = 32 >> step, off = 16 >> step;
        const bool upper = lane & off;
#pragma unroll
        for (int i = 0; i < n; i++) {
            const float mine = upper ? v[i + n] : v[i], theirs = upper ? v[i] : v[i + n];
            v[i] = mine + __shfl_xor_sync(0xffffffffu, theirs, off);
        }
    }
}

constexpr int SUB = 16; /* tokens per sub-chunk */
constexpr int CHUNK_THREADS = 512, CHUNK_WARPS = CHUNK_THREADS / 32;

/* A chunk's rows: none for an idle sequence or one outside the cache (flagged by the scan). */
__device__ __forceinline__ int chunk_rows(const ncb_delta &a, int chunk, int &first) {
    first = a.chunk_first[chunk];
    const int pos = a.conv.pos[first], slot = a.conv.slot_map ? a.conv.slot_map[first] : first;
    return pos < 0 || slot < 0 || slot >= a.conv.n_slots ? 0 : a.chunk_count[chunk];
}
/* Offset of a (chunk, head) in a scratch array of `size` elements each. */
__device__ __forceinline__ size_t scratch_at(const ncb_delta &a, int chunk, int h, int size) { return ((size_t)chunk * a.heads + h) * size; }

template <int MT> __host__ __device__ inline size_t chunk_smem(int D) {
    constexpr int C = SUB * MT;
    return (size_t)3 * C * D * 4 + (size_t)6 * C * (D + 8) * 2 + (size_t)C * (C + 4) * 4 + (size_t)MT * D * 4 + C * 4 + C * sizeof(Place);
}

/* Grid (chunks, heads). C = 16 MT: 64 for dim <= 128, 32 for dim <= 256, so that MT dim <= the block's threads. */
template <int MT> __global__ void __launch_bounds__(CHUNK_THREADS, 1) k_delta_chunk(const ncb_delta a) {
    extern __shared__ __align__(16) uint8_t raw[];
    constexpr int C = SUB * MT, SA = C + 4;
    const int chunk = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t2 = (lane & 3) * 2;
    const int D = a.dim, V = a.vdim, sd = D + 8, kh = h / (a.heads / a.kv_heads);
    float *q = reinterpret_cast<float *>(raw), *k = q + C * D, *al = k + C * D;  /* [C][D] */
    bf16 *qs = reinterpret_cast<bf16 *>(al + C * D), *ks = qs + 2 * C * sd, *kd = ks + 2 * C * sd; /* [2][C][sd] */
    float *A = reinterpret_cast<float *>(kd + 2 * C * sd), *G = A + C * SA, *beta = G + MT * D;
    Place *place = reinterpret_cast<Place *>(beta + C);
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    int first;
    const int n = chunk_rows(a, chunk, first);
    if (n == 0) return;
    const bf16 *proj = (const bf16 *)a.conv.proj;
    for (int i = tid; i < C * SA; i += CHUNK_THREADS) A[i] = 0.f;
    if (tid < C) {
        if (tid < n) place[tid] = place_of(a.conv, first + tid);
        beta[tid] = tid < n ? sigmoid(to_f(proj[(size_t)(first + tid) * a.conv.ldp + a.off_b + h])) : 0.f;
    }
    __syncthreads();
    for (int i = tid; i < C * (D / 2); i += CHUNK_THREADS) {
        const int t = i / (D / 2), d = 2 * (i % (D / 2));
        float2 x = make_float2(0.f, 0.f), y = x;
        if (t < n) {
            x = conv2<bf16>(a.conv, first + t, place[t], a.off_q + kh * D + d);
            y = conv2<bf16>(a.conv, first + t, place[t], a.off_k + kh * D + d);
        }
        *reinterpret_cast<float2 *>(q + t * D + d) = make_float2(silu(x.x), silu(x.y));
        *reinterpret_cast<float2 *>(k + t * D + d) = make_float2(silu(y.x), silu(y.y));
    }
    { /* decays: low-rank products, 8 channels per warp at a time */
        const bf16 *w = (const bf16 *)a.a2_rows + (size_t)h * D * a.rank_a;
        const float a_exp = a.a_exp[h];
        for (int d0 = warp * 8; d0 < D; d0 += CHUNK_WARPS * 8) {
            float acc[MT][4] = {};
            for (int r = 0; r < a.rank_a; r += 16) {
                const bf16 *b = w + (size_t)(d0 + g) * a.rank_a + r + t2;
                const uint32_t b0 = *reinterpret_cast<const uint32_t *>(b), b1 = *reinterpret_cast<const uint32_t *>(b + 8);
#pragma unroll
                for (int m = 0; m < MT; m++) {
                    const int lo = m * 16 + g, hi = lo + 8;
                    const bf16 *x = proj + (size_t)first * a.conv.ldp + a.off_a + r + t2;
                    uint32_t f[4];
                    f[0] = lo < n ? *reinterpret_cast<const uint32_t *>(x + (size_t)lo * a.conv.ldp) : 0u;
                    f[1] = hi < n ? *reinterpret_cast<const uint32_t *>(x + (size_t)hi * a.conv.ldp) : 0u;
                    f[2] = lo < n ? *reinterpret_cast<const uint32_t *>(x + (size_t)lo * a.conv.ldp + 8) : 0u;
                    f[3] = hi < n ? *reinterpret_cast<const uint32_t *>(x + (size_t)hi * a.conv.ldp + 8) : 0u;
                    mma_bf16(acc[m], f, b0, b1);
                }
            }
            const float2 bias = *reinterpret_cast<const float2 *>(a.dt_bias + h * D + d0 + t2);
#pragma unroll
            for (int m = 0; m < MT; m++)
#pragma unroll
                for (int r = 0; r < 2; r++) {
                    const int t = m * 16 + r * 8 + g;
                    *reinterpret_cast<float2 *>(al + t * D + d0 + t2) =
                        t < n ? make_float2(decay_of(acc[m][2 * r] + bias.x, a_exp), decay_of(acc[m][2 * r + 1] + bias.y, a_exp)) : make_float2(1.f, 1.f);
                }
        }
    }
    __syncthreads();
    for (int t = warp; t < C; t += CHUNK_WARPS) { /* unit vectors */
        float x = 0.f, y = 0.f;
        for (int d = lane; d < D; d += 32) x = fmaf(q[t * D + d], q[t * D + d], x), y = fmaf(k[t * D + d], k[t * D + d], y);
        for (int o = 16; o > 0; o >>= 1) x += __shfl_xor_sync(0xffffffffu, x, o), y += __shfl_xor_sync(0xffffffffu, y, o);
        x = a.q_scale / sqrtf(x + UNIT_EPS), y = 1.f / sqrtf(y + UNIT_EPS);
        for (int d = lane; d < D; d += 32) q[t * D + d] *= x, k[t * D + d] *= y;
    }
    __syncthreads();
    for (int i = tid; i < MT * D; i += CHUNK_THREADS) { /* per sub-chunk: q, k with the decays since its start, k with those to its end */
        const int sub = i / D, d = i - sub * D;
        float f = 1.f;
#pragma unroll
        for (int t = 0; t < SUB; t++) {
            const int r = sub * SUB + t;
            f *= al[r * D + d];
            split1(q[r * D + d] * f, qs + r * sd + d, qs + (C + r) * sd + d);
            split1(k[r * D + d] * f, ks + r * sd + d, ks + (C + r) * sd + d);
        }
        G[i] = f;
        f = 1.f;
#pragma unroll
        for (int t = SUB - 1; t >= 0; t--) {
            const int r = sub * SUB + t;
            split1(k[r * D + d] * f, kd + r * sd + d, kd + (C + r) * sd + d);
            f *= al[r * D + d];
        }
    }
    __syncthreads();
    bf16 *B = (bf16 *)a.b_terms + scratch_at(a, chunk, h, 2 * C * C);
    auto put = [&](bool keys, int t, int s, float v) { /* a score of k with k (A, in shared memory), or of q with k (B) */
        if (keys) A[t * SA + s] = beta[t] * v;
        else split1(v, B + t * C + s, B + (C + t) * C + s);
    };
    constexpr int PAIRS = MT * (MT - 1) / 2;
    for (int task = warp; task < 2 * PAIRS; task += CHUNK_WARPS) { /* sub-chunk pairs (i, j), j < i */
        const bool keys = task < PAIRS;
        int i = 1, j = task - (keys ? 0 : PAIRS);
        while (j >= i) j -= i, i++;
        if (i * SUB >= n) continue;
        float acc[2][4] = {};
        const uint32_t xa = smem_addr(keys ? ks : qs) + ((i * SUB + (lane & 15)) * sd + (lane >> 4) * 8) * 2;
        const uint32_t ya = smem_addr(kd) + ((j * SUB + (lane >> 4) * 8 + (lane & 7)) * sd + ((lane >> 3) & 1) * 8) * 2;
        for (int d0 = 0; d0 < D; d0 += 16) {
            uint32_t xh[4], xl[4], yh[4], yl[4];
            ldsm4(xh, xa + d0 * 2);
            ldsm4(xl, xa + (C * sd + d0) * 2);
            ldsm4(yh, ya + d0 * 2);
            ldsm4(yl, ya + (C * sd + d0) * 2);
            if (i - j > 1) {
                float f[4] = {1.f, 1.f, 1.f, 1.f}; /* columns t2, t2 + 1, t2 + 8, t2 + 9 */
                for (int m = j + 1; m < i; m++)
#pragma unroll
                    for (int e = 0; e < 4; e++) f[e] *= G[m * D + d0 + t2 + (e & 1) + (e >> 1) * 8];
                rescale2(xh[0], xl[0], f[0], f[1]), rescale2(xh[1], xl[1], f[0], f[1]);
                rescale2(xh[2], xl[2], f[2], f[3]), rescale2(xh[3], xl[3], f[2], f[3]);
            }
#pragma unroll
            for (int c = 0; c < 2; c++) {
                mma_bf16(acc[c], xh, yh[2 * c], yh[2 * c + 1]);
                mma_bf16(acc[c], xh, yl[2 * c], yl[2 * c + 1]);
                mma_bf16(acc[c], xl, yh[2 * c], yh[2 * c + 1]);
            }
        }
#pragma unroll
        for (int c = 0; c < 2; c++)
#pragma unroll
            for (int e = 0; e < 4; e++) put(keys, i * SUB + g + (e >> 1) * 8, j * SUB + c * 8 + t2 + (e & 1), acc[c][e]);
    }
    for (int task = CHUNK_WARPS - 1 - warp; task < MT * 8; task += CHUNK_WARPS) { /* inside a sub-chunk: (q or k, sub-chunk, four s) */
        const bool keys = task & 1;
        const int i0 = (task >> 3) * SUB, s0 = (task >> 1) % 4 * 4;
        const float *x = keys ? k : q;
        float acc[64]; /* [s][t] */
#pragma unroll
        for (int e = 0; e < 64; e++) acc[e] = 0.f;
        if (i0 < n)
            for (int d = lane; d < D; d += 32) {
                float f[4];
#pragma unroll
                for (int e = 0; e < 4; e++) f[e] = k[(i0 + s0 + e) * D + d];
#pragma unroll
                for (int t = 0; t < SUB; t++) {
                    if (t < s0) continue;
                    const float xt = x[(i0 + t) * D + d], al_t = al[(i0 + t) * D + d];
#pragma unroll
                    for (int e = 0; e < 4; e++) {
                        if (t > s0 + e) f[e] *= al_t;
                        if (t >= s0 + e) acc[e * 16 + t] = fmaf(xt, f[e], acc[e * 16 + t]);
                    }
                }
            }
        reduce64(acc, lane);
#pragma unroll
        for (int e = 0; e < 2; e++) {
            const int s = s0 + (2 * lane + e) / 16, t = (2 * lane + e) % 16;
            if (keys ? t > s : t >= s) put(keys, i0 + t, i0 + s, acc[e]);
            else if (!keys) put(false, i0 + t, i0 + s, 0.f);
        }
    }
    __syncthreads();
    /* Columns: U_0 and W (the solve), k with the decays to the chunk's end, q with those since its start. The values are staged
     * where the terms were, `wide` of them at a time. */
    float *vs = reinterpret_cast<float *>(qs);
    const int wide = 3 * sd / 16 * 16;
    for (int v0 = 0; v0 < V; v0 += wide) {
        const int nv = min(wide, V - v0);
        if (v0) __syncthreads();
        for (int i = tid; i < C * (nv / 2); i += CHUNK_THREADS) {
            const int t = i / (nv / 2), v = 2 * (i % (nv / 2));
            float2 x = make_float2(0.f, 0.f);
            if (t < n) x = conv2<bf16>(a.conv, first + t, place[t], a.off_v + h * V + v0 + v);
            *reinterpret_cast<float2 *>(vs + t * nv + v) = make_float2(beta[t] * silu(x.x), beta[t] * silu(x.y));
        }
        __syncthreads();
        for (int c = tid; c < nv + (v0 ? 0 : 3 * D); c += CHUNK_THREADS) {
            if (c < nv + D) {
                float x[C];
                const int d = c - nv;
                if (d < 0) {
#pragma unroll
                    for (int t = 0; t < C; t++) x[t] = vs[t * nv + c];
                } else {
                    float f = 1.f;
#pragma unroll
                    for (int t = 0; t < C; t++) {
                        f *= al[t * D + d];
                        x[t] = beta[t] * k[t * D + d] * f;
                    }
                }
#pragma unroll
                for (int t = 1; t < C; t++) {
                    float v = x[t], w = 0.f;
#pragma unroll
                    for (int s = 0; s < t; s += 4) {
                        const float4 r = *reinterpret_cast<const float4 *>(A + t * SA + s);
                        v = fmaf(-r.x, x[s], v);
                        if (s + 1 < t) w = fmaf(r.y, x[s + 1], w);
                        if (s + 2 < t) v = fmaf(-r.z, x[s + 2], v);
                        if (s + 3 < t) w = fmaf(r.w, x[s + 3], w);
                    }
                    x[t] = v - w;
                }
                if (d >= 0) {
                    bf16 *w = (bf16 *)a.w_terms + scratch_at(a, chunk, h, 2 * C * D) + d;
#pragma unroll
                    for (int t = 0; t < C; t++) split1(x[t], w + t * D, w + (C + t) * D);
                } else {
                    float4 *u = reinterpret_cast<float4 *>(a.u0 + scratch_at(a, chunk, h, V * C) + (size_t)(v0 + c) * C);
#pragma unroll
                    for (int t = 0; t < C; t += 4) u[t / 4] = make_float4(x[t], x[t + 1], x[t + 2], x[t + 3]);
                }
            } else {
                const bool keys = c < nv + 2 * D;
                const int d = c - nv - (keys ? 1 : 2) * D;
                bf16 *w = (bf16 *)(keys ? a.kd_terms : a.q_terms) + scratch_at(a, chunk, h, 2 * C * D) + d;
                float f = 1.f;
                if (keys) {
#pragma unroll 8
                    for (int t = C - 1; t >= 0; t--) {
                        split1(k[t * D + d] * f, w + t * D, w + (C + t) * D);
                        f *= al[t * D + d];
                    }
                    a.chunk_decay[scratch_at(a, chunk, h, D) + d] = f;
                } else {
#pragma unroll 8
                    for (int t = 0; t < C; t++) {
                        f *= al[t * D + d];
                        split1(q[t * D + d] * f, w + t * D, w + (C + t) * D);
                    }
                }
            }
        }
    }
}

/* Bytes of one stage of k_delta_scan: the terms of W and of k, U_0 of the block's values, the chunk's decay. */
__host__ __device__ inline int scan_stage(int C, int D, int values) { return 4 * C * (D + 8) * 2 + values * (C + 4) * 4 + D * 4; }

/* Grid (ceil(vdim / (16 warps)), heads, segments); a warp owns 16 values. DT = upper bound of dim / 8, C = 64 or 32. */
template <int C, int DT> __global__ void __launch_bounds__(128) k_delta_scan(const ncb_delta a) {
    extern __shared__ __align__(16) uint8_t raw[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t2 = (lane & 3) * 2, threads = blockDim.x, warps = threads / 32;
    const int h = blockIdx.y, seg = blockIdx.z, D = a.dim, V = a.vdim, sd = D + 8, su = C + 4, values = 16 * warps, v0 = blockIdx.x * values;
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const int first = a.seg_first[seg], c0 = a.seg_chunk[seg], c1 = a.seg_chunk[seg + 1];
    const int pos0 = a.conv.pos[first], slot = a.conv.slot_map ? a.conv.slot_map[first] : first;
    if (pos0 < 0 || slot < 0 || slot >= a.conv.n_slots) {
        if (tid == 0 && pos0 >= 0) flag(a.status, NCB_DEV_BAD_POSITION);
        return;
    }
    const int bytes = scan_stage(C, D, values);
    auto fetch = [&](int chunk) {
        const uint32_t dst = smem_addr(raw) + ((chunk - c0) & 1) * bytes;
        const bf16 *w = (const bf16 *)a.w_terms + scratch_at(a, chunk, h, 2 * C * D), *kd = (const bf16 *)a.kd_terms + scratch_at(a, chunk, h, 2 * C * D);
        const int per = D / 8;
        for (int i = tid; i < 2 * C * per; i += threads) {
            const int r = i / per, c = i - r * per;
            cp_async16(dst + (r * sd + c * 8) * 2, w + (size_t)i * 8);
            cp_async16(dst + ((2 * C + r) * sd + c * 8) * 2, kd + (size_t)i * 8);
        }
        const float *u = a.u0 + scratch_at(a, chunk, h, V * C) + (size_t)v0 * C;
        for (int i = tid; i < min(values, V - v0) * (C / 4); i += threads)
            cp_async16(dst + 4 * C * sd * 2 + (i / (C / 4) * su + i % (C / 4) * 4) * 4, u + (size_t)i * 4);
        const float *f = a.chunk_decay + scratch_at(a, chunk, h, D);
        for (int i = tid; i < D / 4; i += threads) cp_async16(dst + 4 * C * sd * 2 + values * su * 4 + i * 16, f + i * 4);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(c0);
    const int mine = v0 + warp * 16, dt = D / 8; /* vdim is a multiple of 16: all of a warp's values or none */
    const bool live = mine < V;
    float *state = a.state + ((size_t)slot * a.heads + h) * D * V + mine + g;
    float s[DT][4]; /* S^T: values g, g + 8; key channels 8 j + t2, + 1 */
#pragma unroll
    for (int j = 0; j < DT; j++)
#pragma unroll
        for (int e = 0; e < 4; e++)
            s[j][e] = live && j < dt && pos0 > 0 ? state[(size_t)(8 * j + t2 + (e & 1)) * V + (e >> 1) * 8] : 0.f;
    for (int chunk = c0; chunk < c1; chunk++) {
        if (chunk + 1 < c1) {
            fetch(chunk + 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        if (live) {
            const uint8_t *stage = raw + ((chunk - c0) & 1) * bytes;
            const uint32_t ws = smem_addr(stage), ks = ws + 2 * C * sd * 2;
            const float *u0 = reinterpret_cast<const float *>(stage + 4 * C * sd * 2) + (warp * 16 + g) * su + t2;
            const float *f = reinterpret_cast<const float *>(stage + 4 * C * sd * 2 + values * su * 4) + t2;
            float u[C / 8][4]; /* U^T: values g, g + 8; tokens 8 j + t2, + 1 */
#pragma unroll
            for (int j = 0; j < C / 8; j++) {
                const float2 lo = *reinterpret_cast<const float2 *>(u0 + 8 * j), hi = *reinterpret_cast<const float2 *>(u0 + 8 * su + 8 * j);
                u[j][0] = lo.x, u[j][1] = lo.y, u[j][2] = hi.x, u[j][3] = hi.y;
            }
            bf16 *st = (bf16 *)a.s_terms + scratch_at(a, chunk, h, 2 * V * D) + (size_t)(mine + g) * D + t2;
            const uint32_t wb = ws + ((lane >> 4) * 8 + (lane & 7)) * sd * 2 + ((lane >> 3) & 1) * 16;
#pragma unroll
            for (int kk = 0; kk < DT / 2; kk++)
                if (2 * kk < dt) {
                    uint32_t hi[4], lo[4];
#pragma unroll
                    for (int e = 0; e < 4; e++) {
                        split2(s[2 * kk + (e >> 1)][2 * (e & 1)], s[2 * kk + (e >> 1)][2 * (e & 1) + 1], hi[e], lo[e]);
                        uint32_t *p = reinterpret_cast<uint32_t *>(st + (size_t)(e & 1) * 8 * D + 16 * kk + (e >> 1) * 8);
                        p[0] = hi[e];
                        p[(size_t)V * D / 2] = lo[e];
                        hi[e] ^= 0x80008000u, lo[e] ^= 0x80008000u; /* U_0 - W S */
                    }
#pragma unroll
                    for (int c = 0; c < C / 16; c++) {
                        uint32_t bh[4], bl[4];
                        ldsm4(bh, wb + (c * 16 * sd + kk * 16) * 2);
                        ldsm4(bl, wb + ((C + c * 16) * sd + kk * 16) * 2);
#pragma unroll
                        for (int e = 0; e < 2; e++) {
                            mma_bf16(u[2 * c + e], hi, bh[2 * e], bh[2 * e + 1]);
                            mma_bf16(u[2 * c + e], hi, bl[2 * e], bl[2 * e + 1]);
                            mma_bf16(u[2 * c + e], lo, bh[2 * e], bh[2 * e + 1]);
                        }
                    }
                }
#pragma unroll
            for (int j = 0; j < DT; j++)
                if (j < dt) {
                    const float2 x = *reinterpret_cast<const float2 *>(f + 8 * j);
                    s[j][0] *= x.x, s[j][1] *= x.y, s[j][2] *= x.x, s[j][3] *= x.y;
                }
            bf16 *ut = (bf16 *)a.u_terms + scratch_at(a, chunk, h, 2 * V * C) + (size_t)(mine + g) * C + t2;
            const uint32_t kb = ks + (lane & 15) * sd * 2 + (lane >> 4) * 16;
#pragma unroll
            for (int kk = 0; kk < C / 16; kk++) {
                uint32_t hi[4], lo[4];
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    split2(u[2 * kk + (e >> 1)][2 * (e & 1)], u[2 * kk + (e >> 1)][2 * (e & 1) + 1], hi[e], lo[e]);
                    uint32_t *p = reinterpret_cast<uint32_t *>(ut + (size_t)(e & 1) * 8 * C + 16 * kk + (e >> 1) * 8);
                    p[0] = hi[e];
                    p[(size_t)V * C / 2] = lo[e];
                }
#pragma unroll
                for (int j = 0; j < DT / 2; j++)
                    if (2 * j < dt) {
                        uint32_t bh[4], bl[4];
                        ldsm4_t(bh, kb + (kk * 16 * sd + j * 16) * 2);
                        ldsm4_t(bl, kb + ((C + kk * 16) * sd + j * 16) * 2);
#pragma unroll
                        for (int e = 0; e < 2; e++) {
                            mma_bf16(s[2 * j + e], hi, bh[2 * e], bh[2 * e + 1]);
                            mma_bf16(s[2 * j + e], hi, bl[2 * e], bl[2 * e + 1]);
                            mma_bf16(s[2 * j + e], lo, bh[2 * e], bh[2 * e + 1]);
                        }
                    }
            }
        }
        __syncthreads(); /* the stage may be overwritten */
    }
    if (live)
#pragma unroll
        for (int j = 0; j < DT; j++)
            if (j < dt)
#pragma unroll
                for (int e = 0; e < 4; e++) state[(size_t)(8 * j + t2 + (e & 1)) * V + (e >> 1) * 8] = s[j][e];
}

constexpr int OUT_THREADS = 256, OUT_WARPS = OUT_THREADS / 32, VT = 16 * OUT_WARPS; /* values a block handles at a time */

template <int MT> __host__ __device__ inline size_t out_smem(int D) {
    constexpr int C = SUB * MT;
    return (size_t)2 * C * (D + 8) * 2 + (size_t)2 * C * (C + 8) * 2 + (size_t)2 * VT * (D + 8) * 2 + (size_t)2 * VT * (C + 8) * 2 + (OUT_WARPS * C + C) * 4;
}

/* Grid (chunks, heads): O = (Q G) S_0 + B U, a warp per 16 values; norm over all values, low-rank gate. */
template <int MT> __global__ void __launch_bounds__(OUT_THREADS, 1) k_delta_out(const ncb_delta a) {
    extern __shared__ __align__(16) uint8_t raw[];
    constexpr int C = SUB * MT, sc = C + 8;
    const int chunk = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t2 = (lane & 3) * 2;
    const int D = a.dim, V = a.vdim, sd = D + 8;
    bf16 *q = reinterpret_cast<bf16 *>(raw), *B = q + 2 * C * sd, *st = B + 2 * C * sc, *ut = st + 2 * VT * sd; /* two terms each */
    float *sums = reinterpret_cast<float *>(ut + 2 * VT * sc), *rstd = sums + OUT_WARPS * C;
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    int first;
    const int n = chunk_rows(a, chunk, first);
    if (n == 0) return;
    auto rows_in = [&](bf16 *dst, int stride, const bf16 *src, int rows, int width) {
        const int per = width / 8;
        for (int i = tid; i < rows * per; i += OUT_THREADS) cp_async16(smem_addr(dst + i / per * stride + i % per * 8), src + (size_t)i * 8);
    };
    rows_in(q, sd, (const bf16 *)a.q_terms + scratch_at(a, chunk, h, 2 * C * D), 2 * C, D);
    rows_in(B, sc, (const bf16 *)a.b_terms + scratch_at(a, chunk, h, 2 * C * C), 2 * C, C);
    for (int i = tid; i < OUT_WARPS * C; i += OUT_THREADS) sums[i] = 0.f;
    const bool direct = V <= VT; /* the whole row of a token is in this block's registers */
    const bf16 *proj = (const bf16 *)a.conv.proj + (size_t)first * a.conv.ldp;
    float acc[MT][2][4];
    for (int v0 = 0; v0 < V; v0 += VT) {
        const int nv = min(VT, V - v0), col0 = warp * 16;
        for (int term = 0; term < 2; term++) {
            rows_in(st + term * VT * sd, sd, (const bf16 *)a.s_terms + scratch_at(a, chunk, h, 2 * V * D) + (size_t)(term * V + v0) * D, nv, D);
            rows_in(ut + term * VT * sc, sc, (const bf16 *)a.u_terms + scratch_at(a, chunk, h, 2 * V * C) + (size_t)(term * V + v0) * C, nv, C);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
#pragma unroll
        for (int i = 0; i < MT * 8; i++) acc[i >> 3][(i >> 2) & 1][i & 3] = 0.f;
        if (col0 < nv) {
            const uint32_t sb = smem_addr(st) + ((col0 + (lane >> 4) * 8 + (lane & 7)) * sd + ((lane >> 3) & 1) * 8) * 2;
            const uint32_t ub = smem_addr(ut) + ((col0 + (lane >> 4) * 8 + (lane & 7)) * sc + ((lane >> 3) & 1) * 8) * 2;
            const uint32_t qb = smem_addr(q) + ((lane & 15) * sd + (lane >> 4) * 8) * 2, bb = smem_addr(B) + ((lane & 15) * sc + (lane >> 4) * 8) * 2;
            for (int k0 = 0; k0 < D; k0 += 16) {
                uint32_t yh[4], yl[4];
                ldsm4(yh, sb + k0 * 2);
                ldsm4(yl, sb + (VT * sd + k0) * 2);
#pragma unroll
                for (int m = 0; m < MT; m++) {
                    uint32_t xh[4], xl[4];
                    ldsm4(xh, qb + (m * 16 * sd + k0) * 2);
                    ldsm4(xl, qb + ((C + m * 16) * sd + k0) * 2);
#pragma unroll
                    for (int c = 0; c < 2; c++) {
                        mma_bf16(acc[m][c], xh, yh[2 * c], yh[2 * c + 1]);
                        mma_bf16(acc[m][c], xh, yl[2 * c], yl[2 * c + 1]);
                        mma_bf16(acc[m][c], xl, yh[2 * c], yh[2 * c + 1]);
                    }
                }
            }
#pragma unroll
            for (int kk = 0; kk < MT; kk++) { /* 16 tokens of the chunk itself; rows before them see none of it */
                uint32_t yh[4], yl[4];
                ldsm4(yh, ub + kk * 32);
                ldsm4(yl, ub + VT * sc * 2 + kk * 32);
#pragma unroll
                for (int m = kk; m < MT; m++) {
                    if (m * 16 >= n) continue; /* rows past the chunk's end have no scores */
                    uint32_t xh[4], xl[4];
                    ldsm4(xh, bb + (m * 16 * sc + kk * 16) * 2);
                    ldsm4(xl, bb + ((C + m * 16) * sc + kk * 16) * 2);
#pragma unroll
                    for (int c = 0; c < 2; c++) {
                        mma_bf16(acc[m][c], xh, yh[2 * c], yh[2 * c + 1]);
                        mma_bf16(acc[m][c], xh, yl[2 * c], yl[2 * c + 1]);
                        mma_bf16(acc[m][c], xl, yh[2 * c], yh[2 * c + 1]);
                    }
                }
            }
#pragma unroll
            for (int m = 0; m < MT; m++)
#pragma unroll
                for (int r = 0; r < 2; r++) {
                    const int t = m * 16 + r * 8 + g;
                    float s = 0.f;
#pragma unroll
                    for (int c = 0; c < 2; c++) {
                        s += acc[m][c][2 * r] * acc[m][c][2 * r] + acc[m][c][2 * r + 1] * acc[m][c][2 * r + 1];
                        if (!direct && t < n)
                            *reinterpret_cast<float2 *>(a.raw + ((size_t)(first + t) * a.heads + h) * V + v0 + col0 + c * 8 + t2) =
                                make_float2(acc[m][c][2 * r], acc[m][c][2 * r + 1]);
                    }
                    s += __shfl_xor_sync(0xffffffffu, s, 1);
                    s += __shfl_xor_sync(0xffffffffu, s, 2);
                    if ((lane & 3) == 0) sums[warp * C + t] += s;
                }
        }
        __syncthreads();
    }
    if (tid < C) {
        float s = 0.f;
        for (int w = 0; w < OUT_WARPS; w++) s += sums[w * C + tid];
        rstd[tid] = 1.f / sqrtf(s / (float)a.norm_count + a.eps);
    }
    __syncthreads();
    for (int v = warp * 16; v < V; v += VT) { /* every thread meets the values that it computed */
        float z[MT][2][4] = {};
        const bf16 *w = (const bf16 *)a.g2_rows + ((size_t)h * V + v + g) * a.rank_g + t2;
        for (int r = 0; r < a.rank_g; r += 16) {
            uint32_t b[2][2];
#pragma unroll
            for (int c = 0; c < 2; c++)
                b[c][0] = *reinterpret_cast<const uint32_t *>(w + (size_t)c * 8 * a.rank_g + r), b[c][1] = *reinterpret_cast<const uint32_t *>(w + (size_t)c * 8 * a.rank_g + r + 8);
#pragma unroll
            for (int m = 0; m < MT; m++) {
                const int lo = m * 16 + g, hi = lo + 8;
                const bf16 *x = proj + a.off_g + r + t2;
                uint32_t f[4];
                f[0] = lo < n ? *reinterpret_cast<const uint32_t *>(x + (size_t)lo * a.conv.ldp) : 0u;
                f[1] = hi < n ? *reinterpret_cast<const uint32_t *>(x + (size_t)hi * a.conv.ldp) : 0u;
                f[2] = lo < n ? *reinterpret_cast<const uint32_t *>(x + (size_t)lo * a.conv.ldp + 8) : 0u;
                f[3] = hi < n ? *reinterpret_cast<const uint32_t *>(x + (size_t)hi * a.conv.ldp + 8) : 0u;
                mma_bf16(z[m][0], f, b[0][0], b[0][1]);
                mma_bf16(z[m][1], f, b[1][0], b[1][1]);
            }
        }
#pragma unroll
        for (int c = 0; c < 2; c++) {
            const float2 weight = *reinterpret_cast<const float2 *>(a.norm + v + c * 8 + t2);
#pragma unroll
            for (int m = 0; m < MT; m++)
#pragma unroll
                for (int r = 0; r < 2; r++) {
                    const int t = m * 16 + r * 8 + g;
                    if (t >= n) continue;
                    float2 o = make_float2(acc[m][c][2 * r], acc[m][c][2 * r + 1]);
                    if (!direct) o = *reinterpret_cast<const float2 *>(a.raw + ((size_t)(first + t) * a.heads + h) * V + v + c * 8 + t2);
                    store2((bf16 *)a.out + (size_t)(first + t) * a.ldo + h * V + v + c * 8 + t2, o.x * rstd[t] * weight.x * sigmoid(z[m][c][2 * r]),
                           o.y * rstd[t] * weight.y * sigmoid(z[m][c][2 * r + 1]));
                }
        }
    }
}

/* ---- host side -------------------------------------------------------------------------------------------------------- */

int check(const ncb_delta &g) {
    const int rc = check_conv(g.conv);
    if (rc != NCB_OK || g.conv.rows == 0) return rc;
    if (g.heads <= 0 || g.heads > 65535 || g.kv_heads <= 0 || g.heads % g.kv_heads || g.dim <= 0 || g.vdim <= 0 || g.dim % 16 || g.vdim % 16 ||
        g.rank_a <= 0 || g.rank_g <= 0 || g.norm_count <= 0 || g.norm_count > g.vdim)
        return NCB_ERR_ARG;
    const int W = g.conv.width;
    if (g.off_q < 0 || g.off_q + g.kv_heads * g.dim > W || g.off_k < 0 || g.off_k + g.kv_heads * g.dim > W || g.off_v < 0 ||
        g.off_v + g.heads * g.vdim > W || (g.off_q | g.off_k | g.off_v) % 2)
        return NCB_ERR_ARG;
    if (g.off_b < 0 || g.off_b + g.heads > g.conv.ldp || g.off_a < 0 || g.off_a + g.rank_a > g.conv.ldp || g.off_g < 0 || g.off_g + g.rank_g > g.conv.ldp)
        return NCB_ERR_ARG;
    if (!g.a2 || !g.g2 || !g.dt_bias || !g.a_exp || !g.norm || !g.state || (g.out && g.ldo < g.heads * g.vdim)) return NCB_ERR_ARG;
    return ((uintptr_t)g.state | (uintptr_t)g.a2 | (uintptr_t)g.g2) % 16 ? NCB_ERR_ALIGN : NCB_OK;
}

template <int NR> int launch_step(const ncb_delta &g, int f32, dim3 grid, size_t smem, int VS, cudaStream_t stream) {
    return f32 ? launch(k_delta_step<float, NR>, grid, STEP_THREADS, smem, (int)grid.x, stream, g, VS)
               : launch(k_delta_step<bf16, NR>, grid, STEP_THREADS, smem, (int)grid.x, stream, g, VS);
}

template <int C, int DT> int launch_scan(const ncb_delta &g, cudaStream_t stream) {
    /* values per block: the fewer, the more SMs take part; blocks of more warps read a chunk's terms less often */
    int warps = 4;
    while (warps > 1 && (long long)((g.vdim + 16 * warps - 1) / (16 * warps)) * g.heads * g.n_segments < 148) warps /= 2;
    const dim3 grid((g.vdim + 16 * warps - 1) / (16 * warps), g.heads, g.n_segments);
    return launch(k_delta_scan<C, DT>, grid, 32 * warps, (size_t)2 * scan_stage(C, g.dim, 16 * warps), 1, stream, g);
}

} /* namespace */

extern "C" {

/* Tokens per chunk of the chunked form for (padded) key size `dim`; 0: only the token-by-token form takes it. */
int delta_chunk_tokens(int dim) { return dim <= 0 ? 0 : dim <= 128 ? 64 : dim <= 256 ? 32 : 0; }

int delta_chunked(const ncb_delta *g, void *stream_ptr) {
    if (!g) return NCB_ERR_ARG;
    int rc = check(*g);
    if (rc != NCB_OK || g->conv.rows == 0) return rc;
    const int C = delta_chunk_tokens(g->dim);
    if (C == 0 || C != g->chunk || g->rank_a % 16 || g->rank_g % 16) return NCB_ERR_UNSUPPORTED;
    if (g->n_chunks <= 0 || g->n_segments <= 0 || g->n_segments > 65535 || !g->seg_first || !g->seg_chunk || !g->chunk_first || !g->chunk_count ||
        !g->a2_rows || !g->g2_rows || !g->w_terms || !g->kd_terms || !g->q_terms || !g->b_terms || !g->u0 || !g->chunk_decay || !g->s_terms ||
        !g->u_terms || (g->out && !g->raw))
        return NCB_ERR_ARG;
    if (((uintptr_t)g->w_terms | (uintptr_t)g->kd_terms | (uintptr_t)g->q_terms | (uintptr_t)g->b_terms | (uintptr_t)g->u0 | (uintptr_t)g->chunk_decay |
         (uintptr_t)g->s_terms | (uintptr_t)g->u_terms | (uintptr_t)g->raw) % 16 || (g->off_a | g->off_g) % 2 || g->ldo % 2)
        return NCB_ERR_ALIGN;
    const cudaStream_t stream = (cudaStream_t)stream_ptr;
    const dim3 grid(g->n_chunks, g->heads);
    rc = C == 64 ? launch(k_delta_chunk<4>, grid, CHUNK_THREADS, chunk_smem<4>(g->dim), 1, stream, *g)
                 : launch(k_delta_chunk<2>, grid, CHUNK_THREADS, chunk_smem<2>(g->dim), 1, stream, *g);
    if (rc != NCB_OK) return rc;
    rc = g->dim <= 64 ? launch_scan<64, 8>(*g, stream) : C == 64 ? launch_scan<64, 16>(*g, stream) : launch_scan<32, 32>(*g, stream);
    if (rc != NCB_OK || !g->out) return rc;
    return C == 64 ? launch(k_delta_out<4>, grid, OUT_THREADS, out_smem<4>(g->dim), 1, stream, *g)
                   : launch(k_delta_out<2>, grid, OUT_THREADS, out_smem<2>(g->dim), 1, stream, *g);
}

int delta_step(const ncb_delta *g, int f32, void *stream) {
    if (!g) return NCB_ERR_ARG;
    const int rc = check(*g);
    if (rc != NCB_OK || g->conv.rows == 0) return rc;
    const int segments = g->seg_first ? g->n_segments : (int)g->conv.rows;
    if (segments <= 0 || segments > 65535 || (g->seg_first && !g->seg_count)) return NCB_ERR_ARG;
    /* values per block: the most whose state fits the registers; less while the GPU has SMs to spare */
    auto rows_per_thread = [&](int VS) { const int dgs = STEP_THREADS / (VS / 4); return dgs ? (g->dim + dgs - 1) / dgs : 1 << 30; };
    auto slices_of = [&](int VS) { return (g->vdim + VS - 1) / VS; };
    int VS = g->vdim;
    while (VS > 16 && (rows_per_thread(VS) > 16 || (long long)segments * g->heads * slices_of(VS) < 148)) {
        const int next = (VS / 2 + 15) / 16 * 16;
        if (slices_of(next) > 8) break;
        VS = next;
    }
    const int slices = slices_of(VS), nr = rows_per_thread(VS);
    const size_t smem = (size_t)step_smem(g->dim, VS, STEP_THREADS / (VS / 4) ? STEP_THREADS / (VS / 4) : 1, g->rank_a, g->rank_g).total * 4;
    if (slices > 8 || nr > 32 || smem > 200 * 1024) return NCB_ERR_UNSUPPORTED;
    const dim3 grid(slices, g->heads, segments);
    if (nr <= 4) return launch_step<4>(*g, f32, grid, smem, VS, (cudaStream_t)stream);
    if (nr <= 8) return launch_step<8>(*g, f32, grid, smem, VS, (cudaStream_t)stream);
    if (nr <= 16) return launch_step<16>(*g, f32, grid, smem, VS, (cudaStream_t)stream);
    return launch_step<32>(*g, f32, grid, smem, VS, (cudaStream_t)stream);
}

} /* extern "C" */
