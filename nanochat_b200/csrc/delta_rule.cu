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
 *     so U = U_0 - W S_0 with [W | U_0] = T beta [G K | V], T = (I + A)^-1, which needs no state:
 *       k_delta_chunk   (all chunks in parallel) convolutions, unit norms, decays, A, T, W, U_0, and B[t][s] = sum_d q k G_t / G_s;
 *       k_delta_scan    (chunk after chunk) U, and the state S <- G_C S + (K G_C / G)^T U; S^T stays in the accumulators of a
 *                       warp, which owns 16 values of the head, and turns into MMA operands in place;
 *       k_delta_out     (all chunks in parallel) O = (Q G) S_0 + B U, norm, gate.
 *     A decay between two tokens is always a product of the decays between them, never a quotient or a difference of long sums,
 *     so none, however strong, overflows or loses the small ones beside it. Products on the tensor cores take their fp32
 *     operands as two bf16 terms each (three MMAs); the low-rank products have bf16 operands to begin with.
 * T is the type of projections and outputs: bf16, or float for a model that runs in 32-bit.
 */
#include "short_conv.cuh"
#include "umma.cuh"

#include <cooperative_groups.h>

namespace cg = cooperative_groups;

namespace {

constexpr float LOG2E = 1.4426950408889634f, LN2 = 0.6931471805599453f;

__device__ __forceinline__ float sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
/* The activation of the convolutions: at the precision of what they are kept in. */
template <typename T> __device__ __forceinline__ float silu(float z) { return sizeof(T) == 2 ? __fdividef(z, 1.f + ex2(-z * LOG2E)) : z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
/* exp(-a_exp softplus(z)). The second form is a few ulps away from the first: log(1 + e) as a series where 1 + e loses e's bits. */
template <typename T> __device__ __forceinline__ float decay_of(float z, float a_exp) { return expf(-a_exp * softplus(z)); }
template <> __device__ __forceinline__ float decay_of<bf16>(float z, float a_exp) {
    const float e = ex2(-fabsf(z) * LOG2E);
    const float series = e * fmaf(e, fmaf(e, fmaf(e, fmaf(e, 0.2f, -0.25f), 1.f / 3.f), -0.5f), 1.f);
    float log2;
    asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(log2) : "f"(1.f + e));
    return ex2(-a_exp * LOG2E * (fmaxf(z, 0.f) + (e < 0.03125f ? series : log2 * LN2)));
}
constexpr float UNIT_EPS = 1e-6f;

__device__ __forceinline__ uint32_t smem_addr(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }

__device__ __forceinline__ void cp_async16(uint32_t dst, const void *src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}

constexpr int STEP_THREADS = 256, STEP_WARPS = STEP_THREADS / 32;

/* Shared memory of k_delta_step in floats; VS: values per block, dgs: groups of key channels, rank: the larger of the two. */
struct StepSmem {
    int q, k, g, v, low, part, u, sums, weights, total;
};
__host__ __device__ inline StepSmem step_smem(int D, int VS, int dgs, int rank_a, int rank_g, int staged) {
    StepSmem s;
    int at = 0;
    auto take = [&](int n) { const int r = at; at += (n + 3) / 4 * 4; return r; };
    const int wide = D > VS ? D : VS;
    s.q = take(D), s.k = take(D), s.g = take(D), s.v = take(VS), s.low = take(rank_a + rank_g);
    const int low_part = STEP_THREADS * 2 > wide ? STEP_THREADS * 2 : wide; /* partial low-rank products */
    s.part = take(2 * dgs * VS > low_part ? 2 * dgs * VS : low_part);
    s.u = take(2 * VS); /* u, then o */
    s.sums = take(4 * STEP_WARPS + 8);
    s.weights = take(staged ? (rank_a * D + rank_g * VS) / 2 : 0); /* bf16: the low-rank weights */
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
template <typename T, int NR> __global__ void __launch_bounds__(STEP_THREADS, NR > 16 ? 1 : 2) k_delta_step(const ncb_delta a, int VS, int staged) {
    extern __shared__ float sm[];
    __shared__ float block_sum;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y, slices = gridDim.x, rank = blockIdx.x;
    const int D = a.dim, V = a.vdim, v0 = rank * VS, nv = min(VS, V - v0), kh = h / (a.heads / a.kv_heads);
    const int columns = VS / 4, dgs = STEP_THREADS / columns, c = tid % columns, dg = tid / columns;
    const StepSmem L = step_smem(D, VS, dgs, a.rank_a, a.rank_g, staged);
    float *q = sm + L.q, *k = sm + L.k, *g = sm + L.g, *v = sm + L.v, *low = sm + L.low, *part = sm + L.part, *u = sm + L.u, *o = u + VS,
          *sums = sm + L.sums;
    const int first = a.seg_first ? a.seg_first[blockIdx.z] : blockIdx.z, count = a.seg_first ? a.seg_count[blockIdx.z] : 1;
    cg::cluster_group cluster = cg::this_cluster();
    const T *a2 = (const T *)a.a2 + (size_t)h * a.rank_a * D, *g2 = (const T *)a.g2 + (size_t)h * a.rank_g * V + v0;
    int ldg = V;
    if (staged) { /* (bf16) weights depend on nothing: towards shared memory before the dependency wait */
        T *w = reinterpret_cast<T *>(sm + L.weights), *u = w + a.rank_a * D;
        for (int i = tid; i < a.rank_a * D / 8; i += STEP_THREADS) cp_async16(smem_addr(w + i * 8), a2 + (size_t)i * 8);
        const int per = nv / 8;
        for (int i = tid; i < a.rank_g * per; i += STEP_THREADS) {
            const int r = i / per, c = (i - r * per) * 8;
            cp_async16(smem_addr(u + r * VS + c), g2 + (size_t)r * V + c);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        a2 = w, g2 = u, ldg = VS;
    }
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
        asm volatile("cp.async.wait_all;" ::: "memory");
        if (a.out)
            for (int i = tid; i < count * nv; i += STEP_THREADS)
                ((T *)a.out)[(size_t)(first + i / nv) * a.ldo + h * V + v0 + i % nv] = from_f<T>(0.f);
        return;
    }
    const bool keep_qk = a.keep && rank == 0 && h % (a.heads / a.kv_heads) == 0;
    for (int t = 0; t < count; t++) {
        const int row = first + t;
        const T *p = (const T *)a.conv.proj + (size_t)row * a.conv.ldp;
        const Place at = place_of(a.conv, row);
        for (int i = tid; i < D + nv / 2; i += STEP_THREADS) { /* pairs of channels: q, k, v */
            const int which = 2 * i / D, j = which < 2 ? 2 * i - which * D : 2 * i - 2 * D;
            const int ch = which == 0 ? a.off_q + kh * D + j : which == 1 ? a.off_k + kh * D + j : a.off_v + h * V + v0 + j;
            const float2 y = conv2<T>(a.conv, row, at, ch);
            *reinterpret_cast<float2 *>((which == 0 ? q : which == 1 ? k : v) + j) = make_float2(silu<T>(y.x), silu<T>(y.y));
            if (a.keep && (which >= 2 || keep_qk)) keep2<T>(a.conv, row, at, ch);
        }
        for (int i = tid; i < a.rank_a + a.rank_g; i += STEP_THREADS)
            low[i] = to_f(i < a.rank_a ? p[a.off_a + i] : p[a.off_g + i - a.rank_a]);
        if (staged && t == 0) asm volatile("cp.async.wait_group 0;" ::: "memory");
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
            g[d] = decay_of<T>(z, a.a_exp[h]);
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
            low_rank<T>(g2, ldg, a.rank_g, nv, low + a.rank_a, part, tid);
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
/* Two 8-column tiles of (xh + xl) (yh + yl)^T without the lo lo product, the three products in accumulators of their own: one
 * warp's dependent MMAs would wait for each other. */
__device__ __forceinline__ void three_terms(float (&acc)[3][2][4], const uint32_t *xh, const uint32_t *xl, const uint32_t *yh, const uint32_t *yl) {
#pragma unroll
    for (int c = 0; c < 2; c++) {
        mma_bf16(acc[0][c], xh, yh[2 * c], yh[2 * c + 1]);
        mma_bf16(acc[1][c], xh, yl[2 * c], yl[2 * c + 1]);
        mma_bf16(acc[2][c], xl, yh[2 * c], yh[2 * c + 1]);
    }
}
__device__ __forceinline__ void ldsm4(uint32_t *r, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4_t(uint32_t *r, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
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
/* Two fp32 operations as one instruction. */
__device__ __forceinline__ float2 mul2(float2 a, float2 b) {
    float2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(reinterpret_cast<uint64_t &>(r)) : "l"(reinterpret_cast<uint64_t &>(a)), "l"(reinterpret_cast<uint64_t &>(b)));
    return r;
}
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
    float2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(reinterpret_cast<uint64_t &>(r))
        : "l"(reinterpret_cast<uint64_t &>(a)), "l"(reinterpret_cast<uint64_t &>(b)), "l"(reinterpret_cast<uint64_t &>(c)));
    return r;
}
/* v[0 .. 63] summed over each half of the warp by halving: lane l of a half ends up with the sums of values 4 l .. 4 l + 3. */
__device__ __forceinline__ void reduce64(float (&v)[64], int lane) {
#pragma unroll
    for (int step = 0; step < 4; step++) {
        const int n = 32 >> step, off = 8 >> step;
        const bool upper = lane & off;
#pragma unroll
        for (int i = 0; i < n; i++) {
            const float mine = upper ? v[i + n] : v[i], theirs = upper ? v[i] : v[i + n];
            v[i] = mine + __shfl_xor_sync(0xffffffffu, theirs, off);
        }
    }
}

constexpr int MAX_SMEM = 226 * 1024;
constexpr int SUB = 16;     /* tokens per sub-chunk */
constexpr int VALUES = 128; /* values k_delta_chunk works on at a time */
#ifndef WIDE_CHUNK_DIM
#define WIDE_CHUNK_DIM 128
#endif

/* A chunk's first row and its place, and how many rows it has: none for an idle sequence or one outside the cache (flagged by the
 * scan). All of this came with the pass's rows, so it may be read before the dependency wait. */
__device__ __forceinline__ int chunk_rows(const ncb_delta &a, int chunk, int &first, Place &at) {
    const int count = a.chunk_count[chunk], within = a.chunk_within[chunk];
    first = a.chunk_first[chunk];
    at = {a.conv.pos[first], a.conv.slot_map ? a.conv.slot_map[first] : first, min(within, a.conv.taps - 1)};
    return at.pos < 0 || at.slot < 0 || at.slot >= a.conv.n_slots ? 0 : count;
}
/* Offset of a (chunk, head) in a scratch array of `size` elements each. */
__device__ __forceinline__ size_t scratch_at(const ncb_delta &a, int chunk, int h, int size) { return ((size_t)chunk * a.heads + h) * size; }

/* Shared memory of k_delta_chunk in bytes: q, k and decays in fp32 [C][D], in their place later the values' terms, T's, and T; terms
 * of q, k [2][C][D + 8] three times, before them the projected rows (with the taps before the chunk) and the low-rank input; A;
 * products of the sub-chunks' decays; beta. */
struct ChunkSmem {
    int al, terms, low, A, G, beta, total;
};
__host__ __device__ inline ChunkSmem chunk_smem(int C, int D, int V, int taps, int rank_a) {
    ChunkSmem s;
    const int fp32 = 3 * C * D * 4, later = 2 * C * (VALUES + 8) * 2 + 2 * C * (C + 8) * 2 + C * (C + 4) * 4;
    s.al = 2 * C * D * 4;
    s.terms = fp32 > later ? fp32 : later;
    const int rows = (C + (taps > CONV_BATCH ? taps : CONV_BATCH) - 1) * (2 * D + (V < VALUES ? V : VALUES)) * 2, staged = rows + C * (rank_a + 8) * 2, terms = 6 * C * (D + 8) * 2;
    s.low = s.terms + rows;
    s.A = s.terms + (staged > terms ? staged : terms);
    s.G = s.A + C * (C + 4) * 4;
    s.beta = s.G + C / SUB * D * 4;
    s.total = s.beta + C * 4;
    return s;
}

/* out[r][c] (16 x 16, stride ldo) = sign * sum over `blocks` 16 x 16 blocks of X . Y, X's blocks side by side (stride SA), Y's one
 * below the other: by thread `i` of `of`. */
template <int SA> __device__ __forceinline__ void block_product(float *out, const float *x, const float *y, int blocks, float sign, int i, int of) {
    for (int e = i; e < SUB * SUB; e += of) {
        const int r = e / SUB, c = e % SUB;
        float v = 0.f;
        for (int k = 0; k < blocks * SUB; k += 4) {
            const float4 a = *reinterpret_cast<const float4 *>(x + r * SA + k);
            v = fmaf(a.x, y[k * SA + c], fmaf(a.y, y[(k + 1) * SA + c], fmaf(a.z, y[(k + 2) * SA + c], fmaf(a.w, y[(k + 3) * SA + c], v))));
        }
        out[r * SA + c] = sign * v;
    }
}

/* Grid (chunks, heads), C = 16 MT tokens. The code runs once per block, so it is kept short: what would be unrolled to thousands
 * of instructions waits for their fetch. */
template <int MT, int CHUNK_THREADS> __global__ void __launch_bounds__(CHUNK_THREADS, 512 / CHUNK_THREADS) k_delta_chunk(const ncb_delta a) {
    extern __shared__ __align__(16) uint8_t raw[];
    constexpr int C = SUB * MT, SA = C + 4, CHUNK_WARPS = CHUNK_THREADS / 32, ST = C + 8, SV = VALUES + 8;
    const int chunk = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t2 = (lane & 3) * 2;
    const int D = a.dim, V = a.vdim, sd = D + 8, kh = h / (a.heads / a.kv_heads);
    const int taps = a.conv.taps, nv0 = min(VALUES, V), wide = 2 * D + nv0; /* staged channels of a row: q, k, the first values */
    const ChunkSmem L = chunk_smem(C, D, V, taps, a.rank_a);
    float *q = reinterpret_cast<float *>(raw), *k = q + C * D, *al = reinterpret_cast<float *>(raw + L.al);
    bf16 *vt = reinterpret_cast<bf16 *>(raw), *tt = vt + 2 * C * SV; /* [2][C][SV], [2][C][ST] */
    float *T = reinterpret_cast<float *>(tt + 2 * C * ST);           /* [C][SA] */
    bf16 *rows = reinterpret_cast<bf16 *>(raw + L.terms), *low = reinterpret_cast<bf16 *>(raw + L.low);
    bf16 *qs = rows, *ks = qs + 2 * C * sd, *kd = ks + 2 * C * sd;   /* [2][C][sd] */
    float *A = reinterpret_cast<float *>(raw + L.A), *G = reinterpret_cast<float *>(raw + L.G), *beta = reinterpret_cast<float *>(raw + L.beta);
    int first;
    Place start;
    const int n = chunk_rows(a, chunk, first, start);
    constexpr int AHEAD = 8; /* 16-wide steps of the decays' weights that are on their way before the dependency wait */
    uint32_t w_ahead[AHEAD][2];
    const bf16 *w_decay = (const bf16 *)a.a2_rows + ((size_t)h * D + warp * 8 + g) * a.rank_a + t2;
#pragma unroll
    for (int i = 0; i < AHEAD; i++)
#pragma unroll
        for (int e = 0; e < 2; e++)
            w_ahead[i][e] = warp * 8 < D && i * 16 < a.rank_a ? *reinterpret_cast<const uint32_t *>(w_decay + i * 16 + e * 8) : 0u;
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    if (n == 0) return;
    const bf16 *proj = (const bf16 *)a.conv.proj;
    /* Fields of the chunk's rows and of the `old` positions before it, a warp per row: n_field runs of `count` channels from
     * ch[field]. Rows past the chunk are its last one; positions before 0 and those that no tap reaches are zeros. */
    const int old = max(taps, CONV_BATCH) - 1;
    auto stage_rows = [&](bf16 *dst, int ld, int n_fields, const int *ch, const int *count) {
        for (int r = warp; r < C + old; r += CHUNK_WARPS) {
            const int t = r - old;
            const bool zero = start.pos + t < 0 || t <= -taps;
            const bf16 *from = t >= -start.before || zero ? proj + (ptrdiff_t)(first + (zero ? 0 : min(t, n - 1))) * a.conv.ldp
                                                          : (const bf16 *)a.conv.ring + ((size_t)start.slot * taps + (start.pos + t) % taps) * a.conv.width;
            bf16 *to = dst + r * ld;
#pragma unroll
            for (int f = 0; f < 3; f++)
                if (f < n_fields) {
                    for (int c = 8 * lane; c < count[f]; c += 256) {
                        if (zero) *reinterpret_cast<uint4 *>(to + c) = make_uint4(0u, 0u, 0u, 0u);
                        else cp_async16(smem_addr(to + c), from + ch[f] + c);
                    }
                    to += count[f];
                }
        }
    };
    /* 8 tokens of a pair of channels from staged rows (x: `old` rows before the first), convolved and activated */
    auto convolve = [&](const bf16 *x, int ld, int ch, float2 (&y)[8]) {
        float2 w[CONV_BATCH], v[8 + CONV_BATCH - 1];
        const float *wp = a.conv.w + (size_t)(taps - 1) * a.conv.width + ch;
#pragma unroll
        for (int back = 0; back < CONV_BATCH; back++)
            w[back] = back < taps ? *reinterpret_cast<const float2 *>(wp - (ptrdiff_t)back * a.conv.width) : make_float2(0.f, 0.f);
        const bf16 *near = x + (old - (CONV_BATCH - 1)) * ld;
#pragma unroll
        for (int i = 0; i < 8 + CONV_BATCH - 1; i++) {
            const uint32_t b = *reinterpret_cast<const uint32_t *>(near + i * ld);
            v[i] = make_float2(__uint_as_float(b << 16), __uint_as_float(b & 0xffff0000u));
        }
#pragma unroll
        for (int t = 0; t < 8; t++) {
            y[t] = mul2(w[0], v[t + CONV_BATCH - 1]);
#pragma unroll
            for (int back = 1; back < CONV_BATCH; back++) y[t] = fma2(w[back], v[t + CONV_BATCH - 1 - back], y[t]);
        }
#pragma unroll 1
        for (int back = CONV_BATCH; back < taps; back++) { /* a longer convolution */
            const float2 f = *reinterpret_cast<const float2 *>(wp - (ptrdiff_t)back * a.conv.width);
#pragma unroll
            for (int t = 0; t < 8; t++) y[t] = fma2(f, load2<bf16>(x + (old + t - back) * ld), y[t]);
        }
#pragma unroll
        for (int t = 0; t < 8; t++) y[t] = make_float2(silu<bf16>(y[t].x), silu<bf16>(y[t].y));
    };
    {
        const int ch[3] = {a.off_q + kh * D, a.off_k + kh * D, a.off_v + h * V}, count[3] = {D, D, nv0};
        stage_rows(rows, wide, 3, ch, count);
    }
    const int sl = a.rank_a + 8;
    for (int t = warp; t < C; t += CHUNK_WARPS)
        for (int c = 8 * lane; c < a.rank_a; c += 256) cp_async16(smem_addr(low + t * sl + c), proj + (size_t)(first + min(t, n - 1)) * a.conv.ldp + a.off_a + c);
    asm volatile("cp.async.commit_group;" ::: "memory");
    for (int i = tid; i < C * SA; i += CHUNK_THREADS) A[i] = 0.f;
    if (tid < C) beta[tid] = tid < n ? sigmoid(to_f(proj[(size_t)(first + tid) * a.conv.ldp + a.off_b + h])) : 0.f;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    for (int i = tid; i < C / 8 * D; i += CHUNK_THREADS) { /* (8 tokens, a pair of channels of q or k) */
        const int d = 2 * (i % D), t0 = i / D * 8, ch = d < D ? a.off_q + kh * D + d : a.off_k + kh * D + d - D;
        float *x = (d < D ? q + d : k + d - D) + t0 * D;
        float2 y[8];
        convolve(rows + t0 * wide + d, wide, ch, y);
#pragma unroll
        for (int t = 0; t < 8; t++) *reinterpret_cast<float2 *>(x + t * D) = t0 + t < n ? y[t] : make_float2(0.f, 0.f);
    }
    /* the first values wait in registers: an item (8 tokens, a pair of values) per thread */
    float2 held[8];
    static_assert(C / 8 * (VALUES / 2) <= CHUNK_THREADS, "one item per thread");
    auto hold_values = [&](const bf16 *x, int ld, int nv, int v0) {
        const int v = 2 * (tid % (nv / 2)), t0 = tid / (nv / 2) * 8;
        if (t0 >= C) return;
        convolve(x + t0 * ld + v, ld, a.off_v + h * V + v0 + v, held);
    };
    auto place_values = [&](int nv) {
        const int v = 2 * (tid % (nv / 2)), t0 = tid / (nv / 2) * 8;
        if (t0 >= C) return;
#pragma unroll
        for (int t = 0; t < 8; t++) { /* (rows past the chunk are finite and meet zero columns of T beta) */
            uint32_t hi, lo;
            split2(held[t].x, held[t].y, hi, lo);
            *reinterpret_cast<uint32_t *>(vt + (t0 + t) * SV + v) = hi;
            *reinterpret_cast<uint32_t *>(vt + (C + t0 + t) * SV + v) = lo;
        }
    };
    hold_values(rows + 2 * D, wide, nv0, 0);
    { /* decays: low-rank products, 8 channels per warp at a time */
        const uint32_t xa = smem_addr(low) + ((lane & 15) * sl + (lane >> 4) * 8) * 2;
        for (int d0 = warp * 8; d0 < D; d0 += CHUNK_WARPS * 8) {
            float acc[MT][4] = {};
            auto step = [&](int r, uint32_t b0, uint32_t b1) {
#pragma unroll
                for (int m = 0; m < MT; m++) {
                    uint32_t f[4];
                    ldsm4(f, xa + (m * 16 * sl + r) * 2);
                    mma_bf16(acc[m], f, b0, b1);
                }
            };
            int r = 0;
            if (d0 == warp * 8) {
#pragma unroll
                for (int i = 0; i < AHEAD; i++, r += 16)
                    if (r < a.rank_a) step(r, w_ahead[i][0], w_ahead[i][1]);
            }
            const bf16 *b = w_decay + (size_t)(d0 - warp * 8) * a.rank_a;
#pragma unroll 4
            for (; r < a.rank_a; r += 16) step(r, *reinterpret_cast<const uint32_t *>(b + r), *reinterpret_cast<const uint32_t *>(b + r + 8));
#pragma unroll
            for (int m = 0; m < MT; m++)
#pragma unroll
                for (int r = 0; r < 2; r++) *reinterpret_cast<float2 *>(al + (m * 16 + r * 8 + g) * D + d0 + t2) = make_float2(acc[m][2 * r], acc[m][2 * r + 1]);
        }
    }
    __syncthreads();
#pragma unroll 1
    for (int t = warp; t < C; t += 4 * CHUNK_WARPS) { /* decays and unit vectors, four tokens at a time */
        const float a_exp = a.a_exp[h];
        float x[4] = {}, y[4] = {};
        for (int d = lane; d < D; d += 32) {
            const float bias = a.dt_bias[h * D + d];
#pragma unroll
            for (int j = 0; j < 4; j++) {
                const int token = t + j * CHUNK_WARPS, r = min(token, C - 1) * D + d;
                x[j] = fmaf(q[r], q[r], x[j]), y[j] = fmaf(k[r], k[r], y[j]);
                if (token < C) al[r] = token < n ? decay_of<bf16>(al[r] + bias, a_exp) : 1.f;
            }
        }
#pragma unroll
        for (int j = 0; j < 4; j++) {
            for (int o = 16; o > 0; o >>= 1) x[j] += __shfl_xor_sync(0xffffffffu, x[j], o), y[j] += __shfl_xor_sync(0xffffffffu, y[j], o);
            x[j] = a.q_scale / sqrtf(x[j] + UNIT_EPS), y[j] = 1.f / sqrtf(y[j] + UNIT_EPS);
        }
        for (int d = lane; d < D; d += 32)
#pragma unroll
            for (int j = 0; j < 4; j++)
                if (t + j * CHUNK_WARPS < C) q[(t + j * CHUNK_WARPS) * D + d] *= x[j], k[(t + j * CHUNK_WARPS) * D + d] *= y[j];
    }
    __syncthreads();
    for (int i = tid; i < MT * D; i += CHUNK_THREADS) { /* (pair of channels, sub-chunk, direction) */
        const int d = 2 * (i % (D / 2)), sub = i / (D / 2) % MT;
        const float2 *x = reinterpret_cast<const float2 *>(q + sub * SUB * D + d), *y = reinterpret_cast<const float2 *>(k + sub * SUB * D + d),
                     *f = reinterpret_cast<const float2 *>(al + sub * SUB * D + d);
        const int ld = D / 2, ls = sd / 2, low = C * sd / 2;
        float2 p = make_float2(1.f, 1.f);
        if (i < MT * (D / 2)) { /* q, k with the decays since the sub-chunk's start */
            uint32_t *qo = reinterpret_cast<uint32_t *>(qs + sub * SUB * sd + d), *ko = reinterpret_cast<uint32_t *>(ks + sub * SUB * sd + d);
#pragma unroll 4
            for (int t = 0; t < SUB; t++) {
                p = mul2(p, f[t * ld]);
                const float2 a = mul2(x[t * ld], p), b = mul2(y[t * ld], p);
                uint32_t hi, lo;
                split2(a.x, a.y, hi, lo);
                qo[t * ls] = hi, qo[low + t * ls] = lo;
                split2(b.x, b.y, hi, lo);
                ko[t * ls] = hi, ko[low + t * ls] = lo;
            }
            *reinterpret_cast<float2 *>(G + sub * D + d) = p;
        } else { /* k with the decays to its end */
            uint32_t *ko = reinterpret_cast<uint32_t *>(kd + sub * SUB * sd + d);
#pragma unroll 4
            for (int t = SUB - 1; t >= 0; t--) {
                const float2 b = mul2(y[t * ld], p);
                uint32_t hi, lo;
                split2(b.x, b.y, hi, lo);
                ko[t * ls] = hi, ko[low + t * ls] = lo;
                p = mul2(p, f[t * ld]);
            }
        }
    }
    __syncthreads();
    bf16 *B = (bf16 *)a.b_terms + scratch_at(a, chunk, h, 2 * C * ST);
    for (int i = tid; i < C * (SUB / 2); i += CHUNK_THREADS) { /* B's diagonal blocks: zero above the diagonal */
        const int t = i / (SUB / 2), s = 2 * (i % (SUB / 2));
        bf16 *p = B + t * ST + t / SUB * SUB;
        if (s > t % SUB) p[s] = p[C * ST + s] = __float2bfloat16_rn(0.f);
        if (s + 1 > t % SUB) p[s + 1] = p[C * ST + s + 1] = __float2bfloat16_rn(0.f);
    }
    auto put = [&](bool keys, int t, int s, float v) { /* a score of k with k (A, in shared memory), or of q with k (B) */
        if (keys) A[t * SA + s] = beta[t] * v;
        else split1(v, B + t * ST + s, B + (C + t) * ST + s);
    };
    constexpr int PAIRS = MT * (MT - 1) / 2;
    for (int task = warp; task < 2 * PAIRS; task += CHUNK_WARPS) { /* sub-chunk pairs (i, j), j < i */
        const bool keys = task < PAIRS;
        int i = 1, j = task - (keys ? 0 : PAIRS);
        while (j >= i) j -= i, i++;
        if (i * SUB >= n) continue;
        float acc[3][2][4] = {};
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
            three_terms(acc, xh, xl, yh, yl);
        }
#pragma unroll
        for (int c = 0; c < 2; c++)
#pragma unroll
            for (int e = 0; e < 4; e++)
                put(keys, i * SUB + g + (e >> 1) * 8, j * SUB + c * 8 + t2 + (e & 1), acc[0][c][e] + acc[1][c][e] + acc[2][c][e]);
    }
    for (int task = CHUNK_WARPS - 1 - warp; task < MT * 4; task += CHUNK_WARPS) { /* inside a sub-chunk: (sub-chunk, four s), k in half a warp, q in the other */
        const bool keys = lane < 16;
        const int i0 = (task >> 2) * SUB, s0 = task % 4 * 4;
        const float *x = keys ? k : q;
        float2 sums[2][SUB]; /* [pair of s][t - s0]: what lies before s is never used */
#pragma unroll
        for (int e = 0; e < 2 * SUB; e++) sums[e / SUB][e % SUB] = make_float2(0.f, 0.f);
        if (i0 < n)
#pragma unroll 1
            for (int d = lane & 15; d < D; d += 16) {
                const float *kp = k + (i0 + s0) * D + d, *xp = x + (i0 + s0) * D + d, *ap = al + (i0 + s0) * D + d;
                float2 f[2] = {make_float2(kp[0], kp[D]), make_float2(kp[2 * D], kp[3 * D])};
#pragma unroll
                for (int t = 0; t < SUB; t++) {
                    if (s0 + t >= SUB) continue;
                    const float xt = xp[t * D], al_t = ap[t * D];
#pragma unroll
                    for (int e = 0; e < 2; e++) { /* s = 2 e, 2 e + 1: decays after s */
                        if (t > 2 * e) f[e] = mul2(f[e], make_float2(al_t, t > 2 * e + 1 ? al_t : 1.f));
                        if (t >= 2 * e) sums[e][t] = fma2(make_float2(xt, xt), f[e], sums[e][t]);
                    }
                }
            }
        float acc[64]; /* [s][t - s0] */
#pragma unroll
        for (int e = 0; e < 2 * SUB; e++) acc[e / SUB * 2 * SUB + e % SUB] = sums[e / SUB][e % SUB].x, acc[(e / SUB * 2 + 1) * SUB + e % SUB] = sums[e / SUB][e % SUB].y;
        reduce64(acc, lane);
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int at = 4 * (lane & 15) + e, s = s0 + at / 16, t = s0 + at % 16;
            if (t < SUB && (keys ? t > s : t >= s)) put(keys, i0 + t, i0 + s, acc[e]);
        }
    }
    __syncthreads();
    place_values(nv0);
    /* T = (I + A)^-1 by blocks of 16: the diagonal's, then T_ij = -T_ii sum_(j <= m < i) A_im T_mj, with the sum in the place of
     * block (j, i). Meanwhile the other warps take the terms over to the whole chunk. */
    if (tid < C) { /* column c of a diagonal block, upwards from its unit */
        const int i0 = tid / SUB * SUB, c = tid % SUB;
        float x[SUB];
#pragma unroll
        for (int r = 0; r < SUB; r++) {
            float v = r == c ? 1.f : 0.f;
#pragma unroll
            for (int m = 0; m < r; m++) v = fmaf(-A[(i0 + r) * SA + i0 + m], x[m], v);
            x[r] = v;
        }
#pragma unroll
        for (int r = 0; r < SUB; r++) T[(i0 + r) * SA + i0 + c] = x[r];
    } else {
        const bf16 *terms[3] = {qs, ks, kd};
        bf16 *out[2] = {(bf16 *)a.q_terms + scratch_at(a, chunk, h, 2 * C * sd), (bf16 *)a.kd_terms + scratch_at(a, chunk, h, 2 * C * sd)};
        for (int i = tid - C; i < 3 * MT * (D / 2); i += CHUNK_THREADS - C) { /* (which, sub-chunk, a pair of channels) */
            const int which = i / (MT * (D / 2)), sub = i / (D / 2) % MT, d = 2 * (i % (D / 2));
            float f0 = 1.f, f1 = 1.f;
            for (int m = which < 2 ? 0 : sub + 1; m < (which < 2 ? sub : MT); m++) f0 *= G[m * D + d], f1 *= G[m * D + d + 1];
            const uint32_t *x = reinterpret_cast<const uint32_t *>(terms[which] + sub * SUB * sd + d);
            uint32_t *y = which == 1 ? const_cast<uint32_t *>(x) : reinterpret_cast<uint32_t *>(out[which / 2] + sub * SUB * sd + d);
            const int ld = sd / 2, low = C * ld;
#pragma unroll 4
            for (int t = 0; t < SUB; t++) {
                uint32_t hi = x[t * ld], lo = x[low + t * ld];
                rescale2(hi, lo, f0, f1);
                y[t * ld] = hi, y[low + t * ld] = lo;
            }
        }
        for (int d = tid - C; d < D; d += CHUNK_THREADS - C) {
            float f = 1.f;
            for (int m = 0; m < MT; m++) f *= G[m * D + d];
            a.chunk_decay[scratch_at(a, chunk, h, D) + d] = f;
        }
    }
    __syncthreads();
#pragma unroll 1
    for (int gap = 1; gap < MT; gap++) { /* block pairs (j + gap, j); 128 threads each */
        const int per = gap == 1 ? 128 : 256, j = tid / per, i = j + gap; /* threads per pair: 128 x 3, 256 x 2, 256 */
        float *sum = T + j * SUB * SA + i * SUB;
        if (i < MT) block_product<SA>(sum, A + i * SUB * SA + j * SUB, T + j * SUB * SA + j * SUB, gap, 1.f, tid % per, per);
        __syncthreads();
        if (i < MT) block_product<SA>(T + i * SUB * SA + j * SUB, T + i * SUB * SA + i * SUB, sum, 1, -1.f, tid % per, per);
        __syncthreads();
    }
    for (int i = tid; i < C * C / 2; i += CHUNK_THREADS) { /* the terms of T beta, zero above the diagonal */
        const int t = i / (C / 2), c = 2 * (i % (C / 2));
        uint32_t hi, lo;
        split2(c <= t ? T[t * SA + c] * beta[c] : 0.f, c + 1 <= t ? T[t * SA + c + 1] * beta[c + 1] : 0.f, hi, lo);
        *reinterpret_cast<uint32_t *>(tt + t * ST + c) = hi;
        *reinterpret_cast<uint32_t *>(tt + (C + t) * ST + c) = lo;
    }
    for (int v0 = 0; v0 < V; v0 += VALUES) {
        const int nv = min(VALUES, V - v0);
        if (v0) { /* more values: their rows where qs was */
            const int ch[3] = {a.off_v + h * V + v0, 0, 0}, count[3] = {nv, 0, 0};
            stage_rows(rows, nv, 1, ch, count);
            asm volatile("cp.async.commit_group;" ::: "memory");
            asm volatile("cp.async.wait_group 0;" ::: "memory");
            __syncthreads();
            hold_values(rows, nv, nv, v0);
            place_values(nv);
        }
        __syncthreads();
        /* U_0^T = V^T (T beta)^T, 16 values per warp; once, W = (T beta) (G K), 16 channels per warp */
        const int n_u = nv / 16, n_w = v0 ? 0 : D / 16;
        for (int task = warp; task < n_u + n_w; task += CHUNK_WARPS) {
            const bool values = task < n_u;
            const int c0 = (values ? task : task - n_u) * 16;
            const uint32_t ta = smem_addr(tt), xb = smem_addr(values ? vt : ks);
#pragma unroll 1
            for (int m = 0; m < MT; m++) { /* 16 tokens of the result */
                float acc[3][2][4] = {};
#pragma unroll 1
                for (int kk = 0; kk <= m; kk++) {
                    uint32_t th[4], tl[4], xh[4], xl[4];
                    if (values) { /* A: values by tokens, from [token][value]; B: T's rows */
                        const uint32_t tb = ta + ((m * 16 + (lane >> 4) * 8 + (lane & 7)) * ST + kk * 16 + ((lane >> 3) & 1) * 8) * 2;
                        const uint32_t at = xb + ((kk * 16 + (lane >> 4) * 8 + (lane & 7)) * SV + c0 + ((lane >> 3) & 1) * 8) * 2;
                        ldsm4_t(xh, at);
                        ldsm4_t(xl, at + C * SV * 2);
                        ldsm4(th, tb);
                        ldsm4(tl, tb + C * ST * 2);
                        three_terms(acc, xh, xl, th, tl);
                    } else { /* A: T's rows; B: channels, from [token][channel] */
                        const uint32_t at = xb + ((kk * 16 + (lane & 15)) * sd + c0 + (lane >> 4) * 8) * 2;
                        const uint32_t tb = ta + ((m * 16 + (lane & 15)) * ST + kk * 16 + (lane >> 4) * 8) * 2;
                        ldsm4_t(xh, at);
                        ldsm4_t(xl, at + C * sd * 2);
                        ldsm4(th, tb);
                        ldsm4(tl, tb + C * ST * 2);
                        three_terms(acc, th, tl, xh, xl);
                    }
                }
#pragma unroll
                for (int c = 0; c < 2; c++)
#pragma unroll
                    for (int r = 0; r < 2; r++) {
                        const float x = acc[0][c][2 * r] + acc[1][c][2 * r] + acc[2][c][2 * r], y = acc[0][c][2 * r + 1] + acc[1][c][2 * r + 1] + acc[2][c][2 * r + 1];
                        if (values) {
                            *reinterpret_cast<float2 *>(a.u0 + scratch_at(a, chunk, h, V * SA) + (size_t)(v0 + c0 + g + r * 8) * SA + m * 16 + c * 8 + t2) = make_float2(x, y);
                        } else {
                            uint32_t hi, lo, *w = reinterpret_cast<uint32_t *>((bf16 *)a.w_terms + scratch_at(a, chunk, h, 2 * C * sd) + (m * 16 + r * 8 + g) * sd + c0 + c * 8 + t2);
                            split2(x, y, hi, lo);
                            w[0] = hi, w[C * sd / 2] = lo;
                        }
                    }
            }
        }
        __syncthreads();
    }
}

/* Bytes of one stage of k_delta_scan: the terms of W and of k, U_0 of the block's values, the chunk's decay. */
__host__ __device__ inline int scan_stage(int C, int D, int values) { return 4 * C * (D + 8) * 2 + values * (C + 4) * 4 + D * 4; }

/* Grid (ceil(vdim / (16 warps)), heads, segments); a warp owns 16 values. DT = upper bound of dim / 8, C = 64 or 32. A chunk's
 * operands lie in memory as they do in shared memory, padded rows and all: four bulk copies, two stages. */
template <int C, int DT> __global__ void __launch_bounds__(128) k_delta_scan(const ncb_delta a) {
    extern __shared__ __align__(16) uint8_t raw[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t2 = (lane & 3) * 2, threads = blockDim.x, warps = threads / 32;
    const int h = blockIdx.y, seg = blockIdx.z, D = a.dim, V = a.vdim, sd = D + 8, su = C + 4, sc = C + 8, values = 16 * warps, v0 = blockIdx.x * values;
    const int bytes = scan_stage(C, D, values), held = min(values, V - v0);
    const uint32_t bars = smem_u32(raw) + 2 * bytes;
    if (tid == 0) {
        mbar_init(bars, 1), mbar_init(bars + 8, 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const int first = a.seg_first[seg], c0 = a.seg_chunk[seg], c1 = a.seg_chunk[seg + 1];
    const int pos0 = a.conv.pos[first], slot = a.conv.slot_map ? a.conv.slot_map[first] : first;
    if (pos0 < 0 || slot < 0 || slot >= a.conv.n_slots) {
        if (tid == 0 && pos0 >= 0) flag(a.status, NCB_DEV_BAD_POSITION);
        return;
    }
    auto fetch = [&](int chunk) { /* one thread */
        const int buf = (chunk - c0) & 1, terms = 2 * C * sd;
        const uint32_t dst = smem_u32(raw) + buf * bytes, bar = bars + 8 * buf;
        mbar_expect_tx(bar, 2 * terms * 2 + held * su * 4 + D * 4);
        bulk_load(dst, (const bf16 *)a.w_terms + scratch_at(a, chunk, h, terms), terms * 2, bar);
        bulk_load(dst + terms * 2, (const bf16 *)a.kd_terms + scratch_at(a, chunk, h, terms), terms * 2, bar);
        bulk_load(dst + 2 * terms * 2, a.u0 + scratch_at(a, chunk, h, V * su) + (size_t)v0 * su, held * su * 4, bar);
        bulk_load(dst + 2 * terms * 2 + values * su * 4, a.chunk_decay + scratch_at(a, chunk, h, D), D * 4, bar);
    };
    if (tid == 0) fetch(c0);
    const int mine = v0 + warp * 16, dt = D / 8; /* vdim is a multiple of 16: all of a warp's values or none */
    const bool live = mine < V;
    float *state = a.state + ((size_t)slot * a.heads + h) * D * V + mine + g;
    float s[DT][4]; /* S^T: values g, g + 8; key channels 8 j + t2, + 1 */
#pragma unroll
    for (int j = 0; j < DT; j++)
#pragma unroll
        for (int e = 0; e < 4; e++)
            s[j][e] = live && j < dt && pos0 > 0 ? state[(size_t)(8 * j + t2 + (e & 1)) * V + (e >> 1) * 8] : 0.f;
    bool ok = true;
    __syncthreads(); /* the barriers exist */
    for (int chunk = c0; chunk < c1; chunk++) {
        if (tid == 0 && chunk + 1 < c1) fetch(chunk + 1);
        const int buf = (chunk - c0) & 1;
        if (!mbar_wait(bars + 8 * buf, ((chunk - c0) >> 1) & 1)) ok = false;
        __syncwarp();
        if (live) {
            const uint8_t *stage = raw + buf * bytes;
            const uint32_t ws = smem_u32(stage), ks = ws + 2 * C * sd * 2;
            const float *u0 = reinterpret_cast<const float *>(stage + 4 * C * sd * 2) + (warp * 16 + g) * su + t2;
            const float *f = reinterpret_cast<const float *>(stage + 4 * C * sd * 2 + values * su * 4) + t2;
            float u[C / 8][4]; /* U^T: values g, g + 8; tokens 8 j + t2, + 1 */
#pragma unroll
            for (int j = 0; j < C / 8; j++) {
                const float2 lo = *reinterpret_cast<const float2 *>(u0 + 8 * j), hi = *reinterpret_cast<const float2 *>(u0 + 8 * su + 8 * j);
                u[j][0] = lo.x, u[j][1] = lo.y, u[j][2] = hi.x, u[j][3] = hi.y;
            }
            uint32_t *st = reinterpret_cast<uint32_t *>((bf16 *)a.s_terms + scratch_at(a, chunk, h, 2 * V * sd) + (size_t)(mine + g) * sd + t2);
            const uint32_t wb = ws + ((lane >> 4) * 8 + (lane & 7)) * sd * 2 + ((lane >> 3) & 1) * 16;
#pragma unroll
            for (int kk = 0; kk < DT / 2; kk++)
                if (2 * kk < dt) {
                    uint32_t hi[4], lo[4], b[C / 16][4];
#pragma unroll
                    for (int c = 0; c < C / 16; c++) ldsm4(b[c], wb + (c * 16 * sd + kk * 16) * 2);
#pragma unroll
                    for (int e = 0; e < 4; e++) {
                        split2(s[2 * kk + (e >> 1)][2 * (e & 1)], s[2 * kk + (e >> 1)][2 * (e & 1) + 1], hi[e], lo[e]);
                        uint32_t *p = st + ((e & 1) * 8 * sd + 16 * kk + (e >> 1) * 8) / 2;
                        p[0] = hi[e];
                        p[(size_t)V * sd / 2] = lo[e];
                        hi[e] ^= 0x80008000u, lo[e] ^= 0x80008000u; /* U_0 - W S */
                    }
#pragma unroll
                    for (int c = 0; c < C / 8; c++) mma_bf16(u[c], hi, b[c / 2][2 * (c & 1)], b[c / 2][2 * (c & 1) + 1]);
#pragma unroll
                    for (int c = 0; c < C / 8; c++) mma_bf16(u[c], lo, b[c / 2][2 * (c & 1)], b[c / 2][2 * (c & 1) + 1]);
#pragma unroll
                    for (int c = 0; c < C / 16; c++) ldsm4(b[c], wb + ((C + c * 16) * sd + kk * 16) * 2);
#pragma unroll
                    for (int c = 0; c < C / 8; c++) mma_bf16(u[c], hi, b[c / 2][2 * (c & 1)], b[c / 2][2 * (c & 1) + 1]);
                }
#pragma unroll
            for (int j = 0; j < DT; j++)
                if (j < dt) {
                    const float2 x = *reinterpret_cast<const float2 *>(f + 8 * j);
                    s[j][0] *= x.x, s[j][1] *= x.y, s[j][2] *= x.x, s[j][3] *= x.y;
                }
            uint32_t *ut = reinterpret_cast<uint32_t *>((bf16 *)a.u_terms + scratch_at(a, chunk, h, 2 * V * sc) + (size_t)(mine + g) * sc + t2);
            const uint32_t kb = ks + (lane & 15) * sd * 2 + (lane >> 4) * 16;
            constexpr int JG = DT / 2 < 4 ? DT / 2 : 4; /* 16-channel groups whose operands are held together */
#pragma unroll
            for (int kk = 0; kk < C / 16; kk++) {
                uint32_t hi[4], lo[4];
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    split2(u[2 * kk + (e >> 1)][2 * (e & 1)], u[2 * kk + (e >> 1)][2 * (e & 1) + 1], hi[e], lo[e]);
                    uint32_t *p = ut + ((e & 1) * 8 * sc + 16 * kk + (e >> 1) * 8) / 2;
                    p[0] = hi[e];
                    p[(size_t)V * sc / 2] = lo[e];
                }
#pragma unroll
                for (int j0 = 0; j0 < DT / 2; j0 += JG)
                    if (2 * j0 < dt) {
                        uint32_t b[JG][4];
#pragma unroll
                        for (int j = 0; j < JG; j++) ldsm4_t(b[j], kb + (kk * 16 * sd + (2 * (j0 + j) < dt ? j0 + j : 0) * 16) * 2);
#pragma unroll
                        for (int e = 0; e < 2 * JG; e++)
                            if (2 * j0 + e < dt) mma_bf16(s[2 * j0 + e], hi, b[e / 2][2 * (e & 1)], b[e / 2][2 * (e & 1) + 1]);
#pragma unroll
                        for (int e = 0; e < 2 * JG; e++)
                            if (2 * j0 + e < dt) mma_bf16(s[2 * j0 + e], lo, b[e / 2][2 * (e & 1)], b[e / 2][2 * (e & 1) + 1]);
#pragma unroll
                        for (int j = 0; j < JG; j++) ldsm4_t(b[j], kb + ((C + kk * 16) * sd + (2 * (j0 + j) < dt ? j0 + j : 0) * 16) * 2);
#pragma unroll
                        for (int e = 0; e < 2 * JG; e++)
                            if (2 * j0 + e < dt) mma_bf16(s[2 * j0 + e], hi, b[e / 2][2 * (e & 1)], b[e / 2][2 * (e & 1) + 1]);
                    }
            }
        }
        __syncthreads(); /* the stage may be overwritten */
    }
    if (!ok && lane == 0) flag(a.status, NCB_DEV_WAIT_TIMEOUT);
    if (live)
#pragma unroll
        for (int j = 0; j < DT; j++)
            if (j < dt)
#pragma unroll
                for (int e = 0; e < 4; e++) state[(size_t)(8 * j + t2 + (e & 1)) * V + (e >> 1) * 8] = s[j][e];
}

constexpr int OUT_THREADS = 512, VT = 128; /* values a block handles at a time: eight column warps of 16, by two halves of the rows */

template <int MT> __host__ __device__ inline size_t out_smem(int D, int rank_g) {
    constexpr int C = SUB * MT;
    return (size_t)2 * C * (D + 8) * 2 + (size_t)2 * C * (C + 8) * 2 + (size_t)2 * VT * (D + 8) * 2 + (size_t)2 * VT * (C + 8) * 2 + (VT / 16 * C + C) * 4 + 16 + (size_t)C * (rank_g + 8) * 2;
}

/* Grid (chunks, heads): O = (Q G) S_0 + B U, a warp per 16 values and half of the rows; norm over all values, low-rank gate (whose
 * product runs while the operands arrive). */
template <int MT> __global__ void __launch_bounds__(OUT_THREADS, 1) k_delta_out(const ncb_delta a) {
    extern __shared__ __align__(16) uint8_t raw[];
    constexpr int C = SUB * MT, sc = C + 8, MH = MT / 2;
    const int chunk = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t2 = (lane & 3) * 2;
    const int D = a.dim, V = a.vdim, sd = D + 8, col0 = (warp & 7) * 16, m0 = (warp >> 3) * MH;
    bf16 *q = reinterpret_cast<bf16 *>(raw), *B = q + 2 * C * sd, *st = B + 2 * C * sc, *ut = st + 2 * VT * sd; /* two terms each */
    float *sums = reinterpret_cast<float *>(ut + 2 * VT * sc), *rstd = sums + VT / 16 * C;
    const uint32_t bars = smem_u32(rstd + C), low = bars + 16; /* the gate's low-rank input [C][rank_g + 8] */
    const int sl = a.rank_g + 8;
    if (tid == 0) {
        mbar_init(bars, 1), mbar_init(bars + 8, 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    int first;
    Place start;
    const int n = chunk_rows(a, chunk, first, start);
    constexpr int AHEAD = 8; /* 16-wide steps of the gate's weights that are on their way before the dependency wait */
    auto gate_weight = [&](int v, int r, int e) { /* (8 values, 8 of the rank) by the bits of e */
        return *reinterpret_cast<const uint32_t *>((const bf16 *)a.g2_rows + ((size_t)h * V + v + g + (e >> 1) * 8) * a.rank_g + r + (e & 1) * 8 + t2);
    };
    uint32_t g_ahead[AHEAD][4];
#pragma unroll
    for (int i = 0; i < AHEAD; i++)
#pragma unroll
        for (int e = 0; e < 4; e++) g_ahead[i][e] = col0 < V && i * 16 < a.rank_g ? gate_weight(col0, i * 16, e) : 0u;
    for (int i = tid; i < VT / 16 * C; i += OUT_THREADS) sums[i] = 0.f;
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    if (n == 0) return;
    const bool direct = V <= VT; /* the whole row of a token is in this block's registers */
    float acc[MH][2][4], z[MH][2][4];
    for (int i = tid; i < C * (a.rank_g / 8); i += OUT_THREADS) {
        const int t = i / (a.rank_g / 8), c = i % (a.rank_g / 8) * 8;
        cp_async16(low + (t * sl + c) * 2, (const bf16 *)a.conv.proj + (size_t)(first + min(t, n - 1)) * a.conv.ldp + a.off_g + c);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    /* the gate's low-rank product for values v .. v + 15 */
    const uint32_t la = low + ((m0 * 16 + (lane & 15)) * sl + (lane >> 4) * 8) * 2;
    auto gate_step = [&](int r, const uint32_t (&b)[4]) {
#pragma unroll
        for (int m = 0; m < MH; m++) {
            uint32_t f[4];
            ldsm4(f, la + (m * 16 * sl + r) * 2);
            mma_bf16(z[m][0], f, b[0], b[1]);
            mma_bf16(z[m][1], f, b[2], b[3]);
        }
    };
    auto gate = [&](int v) {
#pragma unroll
        for (int i = 0; i < MH * 8; i++) z[i >> 3][(i >> 2) & 1][i & 3] = 0.f;
        int r = 0;
        if (v == col0) {
#pragma unroll
            for (int i = 0; i < AHEAD; i++, r += 16)
                if (r < a.rank_g) gate_step(r, g_ahead[i]);
        }
#pragma unroll 4
        for (; r < a.rank_g; r += 16) {
            uint32_t b[4];
#pragma unroll
            for (int e = 0; e < 4; e++) b[e] = gate_weight(v, r, e);
            gate_step(r, b);
        }
    };
    for (int v0 = 0; v0 < V; v0 += VT) {
        const int nv = min(VT, V - v0);
        if (tid == 0) { /* in memory as in shared memory, padded rows and all */
            const bf16 *ss = (const bf16 *)a.s_terms + scratch_at(a, chunk, h, 2 * V * sd) + (size_t)v0 * sd, *us = (const bf16 *)a.u_terms + scratch_at(a, chunk, h, 2 * V * sc) + (size_t)v0 * sc;
            const uint32_t first_bytes = v0 ? 0 : 2 * C * sd * 2, second_bytes = v0 ? 0 : 2 * C * sc * 2;
            mbar_expect_tx(bars, first_bytes + 2 * nv * sd * 2);
            if (!v0) bulk_load(smem_u32(q), (const bf16 *)a.q_terms + scratch_at(a, chunk, h, 2 * C * sd), first_bytes, bars);
            for (int term = 0; term < 2; term++) bulk_load(smem_u32(st + term * VT * sd), ss + (size_t)term * V * sd, nv * sd * 2, bars);
            mbar_expect_tx(bars + 8, second_bytes + 2 * nv * sc * 2);
            if (!v0) bulk_load(smem_u32(B), (const bf16 *)a.b_terms + scratch_at(a, chunk, h, 2 * C * sc), second_bytes, bars + 8);
            for (int term = 0; term < 2; term++) bulk_load(smem_u32(ut + term * VT * sc), us + (size_t)term * V * sc, nv * sc * 2, bars + 8);
        }
        if (!v0) { /* the low-rank input is there, the barriers exist, the sums are zero */
            asm volatile("cp.async.wait_group 0;" ::: "memory");
            __syncthreads();
        }
        const bool live = col0 < nv;
        if (direct && live) gate(col0);
#pragma unroll
        for (int i = 0; i < MH * 8; i++) acc[i >> 3][(i >> 2) & 1][i & 3] = 0.f;
        const uint32_t sb = smem_addr(st) + ((col0 + (lane >> 4) * 8 + (lane & 7)) * sd + ((lane >> 3) & 1) * 8) * 2;
        const uint32_t ub = smem_addr(ut) + ((col0 + (lane >> 4) * 8 + (lane & 7)) * sc + ((lane >> 3) & 1) * 8) * 2;
        const uint32_t qb = smem_addr(q) + ((lane & 15) * sd + (lane >> 4) * 8) * 2, bb = smem_addr(B) + ((lane & 15) * sc + (lane >> 4) * 8) * 2;
        const uint32_t parity = (v0 / VT) & 1;
        bool ok = mbar_wait(bars, parity);
        __syncwarp();
        if (live)
            for (int k0 = 0; k0 < D; k0 += 16) {
                uint32_t yh[4], yl[4];
                ldsm4(yh, sb + k0 * 2);
                ldsm4(yl, sb + (VT * sd + k0) * 2);
                uint32_t xh[MH][4], xl[MH][4];
#pragma unroll
                for (int m = 0; m < MH; m++) {
                    ldsm4(xh[m], qb + ((m0 + m) * 16 * sd + k0) * 2);
                    ldsm4(xl[m], qb + ((C + (m0 + m) * 16) * sd + k0) * 2);
                }
#pragma unroll
                for (int e = 0; e < 3; e++) /* independent accumulators between dependent products */
#pragma unroll
                    for (int m = 0; m < MH; m++)
#pragma unroll
                        for (int c = 0; c < 2; c++) {
                            const uint32_t *y = e == 1 ? yl : yh;
                            mma_bf16(acc[m][c], e == 2 ? xl[m] : xh[m], y[2 * c], y[2 * c + 1]);
                        }
            }
        if (!mbar_wait(bars + 8, parity)) ok = false;
        __syncwarp();
        if (!ok && lane == 0) flag(a.status, NCB_DEV_WAIT_TIMEOUT);
        if (live) {
#pragma unroll
            for (int kk = 0; kk < MT; kk++) { /* 16 tokens of the chunk itself; rows before them see none of it */
                if (kk > m0 + MH - 1) continue;
                uint32_t yh[4], yl[4];
                ldsm4(yh, ub + kk * 32);
                ldsm4(yl, ub + VT * sc * 2 + kk * 32);
#pragma unroll
                for (int m = 0; m < MH; m++) {
                    if (m0 + m < kk || (m0 + m) * 16 >= n) continue; /* rows past the chunk's end have no scores */
                    uint32_t xh[4], xl[4];
                    ldsm4(xh, bb + ((m0 + m) * 16 * sc + kk * 16) * 2);
                    ldsm4(xl, bb + ((C + (m0 + m) * 16) * sc + kk * 16) * 2);
#pragma unroll
                    for (int c = 0; c < 2; c++) {
                        mma_bf16(acc[m][c], xh, yh[2 * c], yh[2 * c + 1]);
                        mma_bf16(acc[m][c], xh, yl[2 * c], yl[2 * c + 1]);
                        mma_bf16(acc[m][c], xl, yh[2 * c], yh[2 * c + 1]);
                    }
                }
            }
#pragma unroll
            for (int m = 0; m < MH; m++)
#pragma unroll
                for (int r = 0; r < 2; r++) {
                    const int t = (m0 + m) * 16 + r * 8 + g;
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
                    if ((lane & 3) == 0) sums[(warp & 7) * C + t] += s;
                }
        }
        __syncthreads();
    }
    if (tid < C) {
        float s = 0.f;
        for (int w = 0; w < VT / 16; w++) s += sums[w * C + tid];
        rstd[tid] = 1.f / sqrtf(s / (float)a.norm_count + a.eps);
    }
    __syncthreads();
    for (int v = col0; v < V; v += VT) { /* every thread meets the values that it computed */
        if (!direct) gate(v);
#pragma unroll
        for (int c = 0; c < 2; c++) {
            const float2 weight = *reinterpret_cast<const float2 *>(a.norm + v + c * 8 + t2);
#pragma unroll
            for (int m = 0; m < MH; m++)
#pragma unroll
                for (int r = 0; r < 2; r++) {
                    const int t = (m0 + m) * 16 + r * 8 + g;
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

template <int NR> int launch_step(const ncb_delta &g, int f32, dim3 grid, size_t smem, int VS, int staged, cudaStream_t stream) {
    return f32 ? launch(k_delta_step<float, NR>, grid, STEP_THREADS, smem, (int)grid.x, stream, g, VS, staged)
               : launch(k_delta_step<bf16, NR>, grid, STEP_THREADS, smem, (int)grid.x, stream, g, VS, staged);
}

template <int C, int DT> int launch_scan(const ncb_delta &g, cudaStream_t stream) {
    /* values per block: the fewer, the more SMs take part; blocks of more warps read a chunk's terms less often */
    int warps = 4;
    while (warps > 1 && (long long)((g.vdim + 16 * warps - 1) / (16 * warps)) * g.heads * g.n_segments < 148) warps /= 2;
    const dim3 grid((g.vdim + 16 * warps - 1) / (16 * warps), g.heads, g.n_segments);
    return launch(k_delta_scan<C, DT>, grid, 32 * warps, (size_t)2 * scan_stage(C, g.dim, 16 * warps) + 16, 1, stream, g);
}

} /* namespace */

extern "C" {

/* Tokens per chunk of the chunked form for these (padded) sizes; 0: only the token-by-token form takes them. */
int delta_chunk_tokens(int dim, int vdim, int taps, int rank_a, int rank_g) {
    if (dim <= 0 || vdim <= 0 || taps <= 0 || rank_a <= 0 || rank_g <= 0) return 0;
    for (int C = dim <= WIDE_CHUNK_DIM ? 64 : 32; C >= 32; C /= 2)
        if (dim <= 256 && (C == 64 ? out_smem<4>(dim, rank_g) : out_smem<2>(dim, rank_g)) <= MAX_SMEM && chunk_smem(C, dim, vdim, taps, rank_a).total <= MAX_SMEM && 2 * scan_stage(C, dim, 64) + 64 <= MAX_SMEM) return C;
    return 0;
}

int delta_chunked(const ncb_delta *g, void *stream_ptr) {
    if (!g) return NCB_ERR_ARG;
    int rc = check(*g);
    if (rc != NCB_OK || g->conv.rows == 0) return rc;
    const int C = delta_chunk_tokens(g->dim, g->vdim, g->conv.taps, g->rank_a, g->rank_g);
    if (C == 0 || C != g->chunk || g->rank_a % 16 || g->rank_g % 16) return NCB_ERR_UNSUPPORTED;
    if (g->n_chunks <= 0 || g->n_segments <= 0 || g->n_segments > 65535 || !g->seg_first || !g->seg_chunk || !g->chunk_first || !g->chunk_count || !g->chunk_within ||
        !g->a2_rows || !g->g2_rows || !g->w_terms || !g->kd_terms || !g->q_terms || !g->b_terms || !g->u0 || !g->chunk_decay || !g->s_terms ||
        !g->u_terms || (g->out && !g->raw))
        return NCB_ERR_ARG;
    if (((uintptr_t)g->w_terms | (uintptr_t)g->kd_terms | (uintptr_t)g->q_terms | (uintptr_t)g->b_terms | (uintptr_t)g->u0 | (uintptr_t)g->chunk_decay |
         (uintptr_t)g->s_terms | (uintptr_t)g->u_terms | (uintptr_t)g->raw) % 16 || (g->off_a | g->off_g | g->off_q | g->off_k | g->off_v | (int)g->conv.ldp | g->conv.width) % 8 || g->ldo % 2)
        return NCB_ERR_ALIGN;
    const cudaStream_t stream = (cudaStream_t)stream_ptr;
    const dim3 grid(g->n_chunks, g->heads);
    const size_t smem = (size_t)chunk_smem(C, g->dim, g->vdim, g->conv.taps, g->rank_a).total;
    rc = C == 64 ? launch(k_delta_chunk<4, 512>, grid, 512, smem, 1, stream, *g)
                 : launch(k_delta_chunk<2, 256>, grid, 256, smem, 1, stream, *g);
    if (rc != NCB_OK) return rc;
    if (C == 64) rc = g->dim <= 64 ? launch_scan<64, 8>(*g, stream) : launch_scan<64, 16>(*g, stream);
    else rc = g->dim <= 64 ? launch_scan<32, 8>(*g, stream) : g->dim <= 128 ? launch_scan<32, 16>(*g, stream) : launch_scan<32, 32>(*g, stream);
    if (rc != NCB_OK || !g->out) return rc;
    return C == 64 ? launch(k_delta_out<4>, grid, OUT_THREADS, out_smem<4>(g->dim, g->rank_g), 1, stream, *g)
                   : launch(k_delta_out<2>, grid, OUT_THREADS, out_smem<2>(g->dim, g->rank_g), 1, stream, *g);
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
    const int dgs = STEP_THREADS / (VS / 4) ? STEP_THREADS / (VS / 4) : 1;
    const int staged = !f32 && (size_t)step_smem(g->dim, VS, dgs, g->rank_a, g->rank_g, 1).total * 4 <= 100 * 1024;
    const size_t smem = (size_t)step_smem(g->dim, VS, dgs, g->rank_a, g->rank_g, staged).total * 4;
    if (slices > 8 || nr > 32 || smem > 200 * 1024) return NCB_ERR_UNSUPPORTED;
    const dim3 grid(slices, g->heads, segments);
    if (nr <= 4) return launch_step<4>(*g, f32, grid, smem, VS, staged, (cudaStream_t)stream);
    if (nr <= 8) return launch_step<8>(*g, f32, grid, smem, VS, staged, (cudaStream_t)stream);
    if (nr <= 16) return launch_step<16>(*g, f32, grid, smem, VS, staged, (cudaStream_t)stream);
    return launch_step<32>(*g, f32, grid, smem, VS, staged, (cudaStream_t)stream);
}

} /* extern "C" */
