/*
 * Gated linear attention with a decay per key channel: per sequence and head a matrix state S [dim][vdim] in fp32,
 *     S_t = diag(alpha_t) S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,   alpha = sigmoid(W_a2 a + b)^(1 / tau),
 * followed by an RMS norm of o over vdim with a weight and a silu output gate. The state lives in one buffer per layer,
 * fp32 [n_slots][heads][dim][vdim]; position 0 starts from zero whatever the slot held before.
 *
 * Two forms, both in fp32 from the projections on:
 *   - k_gla_step: token by token. A block (or a cluster of blocks that share the norm's sum through distributed shared
 *     memory) owns a slice of vdim of one head and streams the state once per token: a decode step, bound by the state's
 *     bytes, and portions of a few tokens;
 *   - chunks of up to 64 tokens (prefill): k_gla_decay (alpha of every row), k_gla_chunk_state (each chunk's own
 *     contribution to the state, all chunks in parallel), k_gla_scan (the states at the chunks' starts, and the sequence's
 *     state at the end), k_gla_chunk_out (outputs of a chunk from its starting state and from itself). Decays between two
 *     tokens are always products of the alphas between them, never quotients or differences of long sums, so no decay,
 *     however strong, overflows or loses the small ones beside it.
 * T is the type of projections and outputs: bf16, or float for a model that runs in 32-bit.
 */
#include "ncb_common.cuh"

#include <cooperative_groups.h>

namespace cg = cooperative_groups;

namespace {

template <typename T> __device__ __forceinline__ float to_f(T v) { return (float)v; }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16_rn(v); }

constexpr float LOG2E = 1.4426950408889634f;

/* log2 of sigmoid(z)^(inv_tau) */
__device__ __forceinline__ float log2_decay(float z, float inv_tau) {
    return (fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * (LOG2E * inv_tau);
}
__device__ __forceinline__ float silu(float z) { return z / (1.f + expf(-z)); }

constexpr int STEP_THREADS = 256;
constexpr int AHEAD_ROWS = 8; /* state rows per thread that are loaded ahead */

/* Grid (slices, heads, segments), cluster (slices, 1, 1); segment z = rows first[z] .. + count[z] - 1 of one slot at
 * ascending positions (first NULL: row z alone). */
template <typename T> __global__ void __launch_bounds__(STEP_THREADS) k_gla_step(const ncb_gla a) {
    extern __shared__ float sm[];
    const int tid = threadIdx.x, h = blockIdx.y, slices = gridDim.x, rank = blockIdx.x;
    const int D = a.dim, V = a.vdim, VS = V / slices, v0 = rank * VS;
    const int groups = VS / 4, dgs = STEP_THREADS / groups;
    float *q = sm, *k = q + D, *alpha = k + D, *part = alpha + D, *o = part + dgs * VS, *sums = o + VS;
    __shared__ float block_sum;
    const int first = a.seg_first ? a.seg_first[blockIdx.z] : blockIdx.z, count = a.seg_first ? a.seg_count[blockIdx.z] : 1;
    cg::cluster_group cluster = cg::this_cluster();
    const int pos0 = a.pos[first], slot = a.slot_map ? a.slot_map[first] : first;
    const bool bad = pos0 >= 0 && (slot < 0 || slot >= a.n_slots);
    float *state = a.state + ((size_t)(bad ? 0 : slot) * a.heads + h) * D * V;
    const int c = tid % groups, dg = tid / groups;
    /* Positions, slots and this state were last written many launches ago (the launch before this one writes the projection
     * alone), so the state's first elements start towards registers before the dependency wait. */
    float4 ahead[AHEAD_ROWS];
#pragma unroll
    for (int i = 0; i < AHEAD_ROWS; i++) {
        const int d = dg + i * dgs;
        ahead[i] = pos0 > 0 && !bad && dg < dgs && d < D ? *reinterpret_cast<const float4 *>(state + (size_t)d * V + v0 + 4 * c)
                                                         : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    if (bad && tid == 0) flag(a.status, NCB_DEV_BAD_POSITION);
    if (pos0 < 0 || bad) { /* an idle row: no state touched, a zero output (every block of the cluster takes this exit) */
        if (a.out)
            for (int i = tid; i < count * VS; i += STEP_THREADS)
                ((T *)a.out)[(size_t)(first + i / VS) * a.ldo + h * V + v0 + i % VS] = from_f<T>(0.f);
        return;
    }
    for (int t = 0; t < count; t++) {
        const int row = first + t;
        const T *p = (const T *)a.proj + (size_t)row * a.ldp;
        for (int d = tid; d < D; d += STEP_THREADS) {
            q[d] = to_f(p[a.off_q + h * D + d]) * a.q_scale;
            k[d] = to_f(p[a.off_k + h * D + d]);
            const float *w = a.a2 + (size_t)(h * D + d) * a.rank;
            float z = a.a2_bias[h * D + d];
            for (int r = 0; r < a.rank; r++) z = fmaf(w[r], to_f(p[a.off_a + r]), z);
            alpha[d] = exp2f(log2_decay(z, a.inv_tau));
        }
        __syncthreads();
        const bool fresh = pos0 + t == 0;
        if (dg < dgs) {
            const T *vp = p + a.off_v + h * V + v0 + 4 * c;
            const float vx = to_f(vp[0]), vy = to_f(vp[1]), vz = to_f(vp[2]), vw = to_f(vp[3]);
            float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
            auto update = [&](int d, float4 s) {
                const float al = alpha[d], kd = k[d], qd = q[d];
                s.x = fmaf(al, s.x, kd * vx), s.y = fmaf(al, s.y, kd * vy);
                s.z = fmaf(al, s.z, kd * vz), s.w = fmaf(al, s.w, kd * vw);
                *reinterpret_cast<float4 *>(state + (size_t)d * V + v0 + 4 * c) = s;
                acc.x = fmaf(qd, s.x, acc.x), acc.y = fmaf(qd, s.y, acc.y);
                acc.z = fmaf(qd, s.z, acc.z), acc.w = fmaf(qd, s.w, acc.w);
            };
            auto stored = [&](int d) {
                return fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4 *>(state + (size_t)d * V + v0 + 4 * c);
            };
            int d = dg;
            if (t == 0) {
#pragma unroll
                for (int i = 0; i < AHEAD_ROWS; i++, d += dgs)
                    if (d < D) update(d, ahead[i]);
            }
#pragma unroll 4
            for (; d < D; d += dgs) update(d, stored(d));
            *reinterpret_cast<float4 *>(part + dg * VS + 4 * c) = acc;
        }
        __syncthreads();
        if (!a.out) continue; /* only the state is wanted */
        float sq = 0.f;
        for (int v = tid; v < VS; v += STEP_THREADS) {
            float s = 0.f;
            for (int j = 0; j < dgs; j++) s += part[j * VS + v];
            o[v] = s;
            sq = fmaf(s, s, sq);
        }
        for (int i = 16; i > 0; i >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, i);
        if ((tid & 31) == 0) sums[tid >> 5] = sq;
        __syncthreads();
        if (tid == 0) {
            float s = 0.f;
            for (int w = 0; w < STEP_THREADS / 32; w++) s += sums[w];
            block_sum = s;
        }
        float total;
        if (slices > 1) {
            cluster.sync();
            total = 0.f;
            for (int s = 0; s < slices; s++) total += *cluster.map_shared_rank(&block_sum, s);
            cluster.sync(); /* nobody overwrites its sum, or leaves, while a peer still reads it */
        } else {
            __syncthreads();
            total = block_sum;
        }
        const float rstd = 1.f / sqrtf(total / (float)a.norm_count + a.eps);
        for (int v = tid; v < VS; v += STEP_THREADS) {
            const float gate = silu(to_f(p[a.off_g + h * V + v0 + v]));
            ((T *)a.out)[(size_t)row * a.ldo + h * V + v0 + v] = from_f<T>(o[v] * rstd * a.norm[v0 + v] * gate);
        }
        __syncthreads();
    }
}

/* ---- chunked form --------------------------------------------------------------------------------------------------- */

constexpr int CHUNK_THREADS = 256;
constexpr int SUB = 16; /* tokens per sub-chunk of the intra-chunk scores */

/* Grid (ceil(rows / DECAY_ROWS), ceil(heads dim / 256)): alpha fp32 [rows][heads dim]; a thread keeps its channel's low-rank
 * weights across the rows. */
constexpr int DECAY_ROWS = 16;
template <typename T> __global__ void __launch_bounds__(CHUNK_THREADS) k_gla_decay(const ncb_gla a) {
    extern __shared__ float sm[]; /* the rows' low-rank inputs, [DECAY_ROWS][rank] */
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const long long first = (long long)blockIdx.x * DECAY_ROWS;
    const int n = (int)(a.rows - first < DECAY_ROWS ? a.rows - first : DECAY_ROWS), HD = a.heads * a.dim;
    for (int i = threadIdx.x; i < n * a.rank; i += CHUNK_THREADS)
        sm[i] = to_f(((const T *)a.proj)[(size_t)(first + i / a.rank) * a.ldp + a.off_a + i % a.rank]);
    __syncthreads();
    const int ch = blockIdx.y * CHUNK_THREADS + threadIdx.x;
    if (ch >= HD) return;
    const float *w = a.a2 + (size_t)ch * a.rank;
    float z[DECAY_ROWS];
#pragma unroll
    for (int t = 0; t < DECAY_ROWS; t++) z[t] = a.a2_bias[ch];
    for (int r = 0; r < a.rank; r++) {
        const float wr = w[r];
#pragma unroll
        for (int t = 0; t < DECAY_ROWS; t++)
            if (t < n) z[t] = fmaf(wr, sm[t * a.rank + r], z[t]);
    }
#pragma unroll
    for (int t = 0; t < DECAY_ROWS; t++)
        if (t < n) a.decay[(size_t)(first + t) * HD + ch] = exp2f(log2_decay(z[t], a.inv_tau));
}

/* acc[4][4] += sum over k of A[k][i0 + i] B[k][j0 + j], both in shared memory with row strides sa and sb. */
__device__ __forceinline__ void tile_fma(float (&acc)[4][4], const float *A, int sa, const float *B, int sb, int kn) {
#pragma unroll 4
    for (int k = 0; k < kn; k++) {
        const float4 x = *reinterpret_cast<const float4 *>(A + k * sa), y = *reinterpret_cast<const float4 *>(B + k * sb);
        const float xa[4] = {x.x, x.y, x.z, x.w}, ya[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
        for (int i = 0; i < 4; i++)
#pragma unroll
            for (int j = 0; j < 4; j++) acc[i][j] = fmaf(xa[i], ya[j], acc[i][j]);
    }
}

/* Grid (chunks, heads, ceil(vdim / 64)): the state a chunk adds, sum_t (k_t alpha_(t+1) .. alpha_end) v_t^T, and its decay. */
template <typename T> __global__ void __launch_bounds__(CHUNK_THREADS) k_gla_chunk_state(const ncb_gla a) {
    extern __shared__ float sm[];
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const int chunk = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * 64, tid = threadIdx.x;
    const int first = a.chunk_first[chunk], n = a.chunk_count[chunk], D = a.dim, V = a.vdim, HD = a.heads * D;
    const int sk = (D + 63) / 64 * 64;
    float *kt = sm, *vt = kt + a.chunk * sk; /* [n][sk], [n][64] */
    for (int d = tid; d < sk; d += CHUNK_THREADS) {
        const float *al = a.decay + (size_t)first * HD + h * D + d;
        const T *kp = (const T *)a.proj + (size_t)first * a.ldp + a.off_k + h * D + d;
        float f = 1.f;
#pragma unroll 8
        for (int t = n - 1; t >= 0; t--) {
            kt[t * sk + d] = d < D ? to_f(kp[(size_t)t * a.ldp]) * f : 0.f;
            if (d < D) f *= al[(size_t)t * HD];
        }
        if (blockIdx.z == 0 && d < D) a.chunk_decay[(size_t)chunk * HD + h * D + d] = f;
    }
    for (int i = tid; i < n * 64; i += CHUNK_THREADS) {
        const int t = i >> 6, v = v0 + (i & 63);
        vt[i] = v < V ? to_f(((const T *)a.proj)[(size_t)(first + t) * a.ldp + a.off_v + h * V + v]) : 0.f;
    }
    __syncthreads();
    float *out = a.states + ((size_t)chunk * a.heads + h) * D * V;
    const int tx = tid & 15, ty = tid >> 4;
    for (int d0 = 0; d0 < D; d0 += 64) {
        float acc[4][4] = {};
        tile_fma(acc, kt + d0 + ty * 4, sk, vt + tx * 4, 64, n);
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const int d = d0 + ty * 4 + i;
            if (d < D && v0 + tx * 4 < V) /* vdim is a multiple of 16 */
                *reinterpret_cast<float4 *>(out + (size_t)d * V + v0 + tx * 4) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
        }
    }
}

/* Grid (heads dim vdim / 4 / 256, segments): states[c] <- the state before chunk c; the slot's state <- the last one. */
__global__ void __launch_bounds__(CHUNK_THREADS) k_gla_scan(const ncb_gla a) {
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const int seg = blockIdx.y, first = a.seg_first[seg], c0 = a.seg_chunk[seg], c1 = a.seg_chunk[seg + 1];
    const int slot = a.slot_map ? a.slot_map[first] : first, pos0 = a.pos[first];
    const size_t total = (size_t)a.heads * a.dim * a.vdim, i = ((size_t)blockIdx.x * CHUNK_THREADS + threadIdx.x) * 4;
    if (i >= total) return;
    if (pos0 < 0 || slot < 0 || slot >= a.n_slots) {
        if (i == 0 && pos0 >= 0) flag(a.status, NCB_DEV_BAD_POSITION);
        return;
    }
    float4 *state = reinterpret_cast<float4 *>(a.state + (size_t)slot * total + i);
    float4 s = pos0 == 0 ? make_float4(0.f, 0.f, 0.f, 0.f) : *state;
    const float *g = a.chunk_decay + i / a.vdim;
    const int HD = a.heads * a.dim;
    constexpr int AHEAD = 8; /* chunks whose loads are in flight together */
    for (int c = c0; c < c1; c += AHEAD) {
        float4 u[AHEAD];
        float f[AHEAD];
#pragma unroll
        for (int j = 0; j < AHEAD; j++)
            if (c + j < c1) {
                u[j] = *reinterpret_cast<const float4 *>(a.states + (size_t)(c + j) * total + i);
                f[j] = g[(size_t)(c + j) * HD];
            }
#pragma unroll
        for (int j = 0; j < AHEAD; j++)
            if (c + j < c1) {
                *reinterpret_cast<float4 *>(a.states + (size_t)(c + j) * total + i) = s;
                s.x = fmaf(f[j], s.x, u[j].x), s.y = fmaf(f[j], s.y, u[j].y);
                s.z = fmaf(f[j], s.z, u[j].z), s.w = fmaf(f[j], s.w, u[j].w);
            }
    }
    *state = s;
}

/* Floats of shared memory k_gla_chunk_out takes. */
__host__ __device__ inline size_t out_floats(int chunk, int D) {
    const int sd = D + 4, sc = chunk + 4;
    return (size_t)3 * chunk * sd + (size_t)SUB * sd + D /* q, k, alpha, scaled q, product so far */
           + (size_t)chunk * sc + (size_t)16 * sc + 16 * 64 + chunk;
}

/* Grid (chunks, heads): o_t = (q_t alpha_1 .. alpha_t) S + sum_(s <= t) A[t][s] v_s with
 * A[t][s] = sum_d q_td k_sd alpha_(s+1)d .. alpha_td, then norm and gate. The chunk is walked in sub-chunks of 16 tokens: inside
 * one, the products run along t for every s; against earlier sub-chunks the decay factors into what q has seen since its
 * sub-chunk began and what k has seen up to there, and k's rows in shared memory are kept at that value as the walk goes on. */
template <typename T> __global__ void __launch_bounds__(CHUNK_THREADS) k_gla_chunk_out(const ncb_gla a) {
    extern __shared__ float sm[];
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const int chunk = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int first = a.chunk_first[chunk], n = a.chunk_count[chunk], D = a.dim, V = a.vdim, HD = a.heads * D, C = a.chunk;
    const int sd = D + 4, sc = C + 4;
    float *q = sm, *k = q + C * sd, *al = k + C * sd, *qs = al + C * sd, *done = qs + SUB * sd;
    float *at = done + D;                      /* scores transposed: [s][t] */
    float *lt = at + C * sc, *rt = lt + 16 * sc; /* staging of the output product: 16 k-values x (t | 64 columns of v) */
    float *ss = rt + 16 * 64;
    const T *proj = (const T *)a.proj;
    for (int i = tid; i < C * D; i += CHUNK_THREADS) {
        const int t = i / D, d = i % D;
        const T *p = proj + (size_t)(first + t) * a.ldp + h * D + d;
        q[t * sd + d] = t < n ? to_f(p[a.off_q]) * a.q_scale : 0.f;
        k[t * sd + d] = t < n ? to_f(p[a.off_k]) : 0.f;
        al[t * sd + d] = t < n ? a.decay[(size_t)(first + t) * HD + h * D + d] : 1.f;
    }
    for (int i = tid; i < C * sc; i += CHUNK_THREADS) at[i] = 0.f;
    for (int d = tid; d < D; d += CHUNK_THREADS) done[d] = 1.f;
    __syncthreads();
    for (int i0 = 0; i0 < n; i0 += SUB) {
        for (int d = tid; d < D; d += CHUNK_THREADS) { /* q with the decays since the sub-chunk's start */
            float f = 1.f;
#pragma unroll
            for (int t = 0; t < SUB; t++) {
                f *= al[(i0 + t) * sd + d];
                qs[t * sd + d] = q[(i0 + t) * sd + d] * f;
            }
        }
        __syncthreads();
        for (int e = tid; e < SUB * i0; e += CHUNK_THREADS) { /* against earlier sub-chunks */
            const int t = e % SUB, s = e / SUB;
            const float4 *x = reinterpret_cast<const float4 *>(qs + t * sd), *y = reinterpret_cast<const float4 *>(k + s * sd);
            float v = 0.f;
            for (int d = 0; d < D / 4; d++) {
                const float4 xv = x[d], yv = y[d];
                v = fmaf(xv.x, yv.x, v), v = fmaf(xv.y, yv.y, v), v = fmaf(xv.z, yv.z, v), v = fmaf(xv.w, yv.w, v);
            }
            at[s * sc + i0 + t] = v;
        }
        { /* inside: thread (s, every 16th channel) runs along t */
            const int s = tid >> 4, lane = tid & 15;
            float acc[SUB];
#pragma unroll
            for (int t = 0; t < SUB; t++) acc[t] = 0.f;
            for (int d = lane; d < D; d += 16) {
                float f = k[(i0 + s) * sd + d];
#pragma unroll
                for (int t = 0; t < SUB; t++) {
                    if (t > s) f *= al[(i0 + t) * sd + d];
                    if (t >= s) acc[t] = fmaf(q[(i0 + t) * sd + d], f, acc[t]);
                }
            }
#pragma unroll
            for (int t = 0; t < SUB; t++) {
                float v = acc[t];
                for (int o = 8; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
                if (lane == t && t >= s) at[(i0 + s) * sc + i0 + t] = v;
            }
        }
        __syncthreads();
        for (int d = tid; d < D; d += CHUNK_THREADS) { /* on to the next sub-chunk */
            const float before = done[d];
            float f = 1.f;
#pragma unroll
            for (int t = SUB - 1; t >= 0; t--) {
                k[(i0 + t) * sd + d] *= f;
                f *= al[(i0 + t) * sd + d];
                q[(i0 + t) * sd + d] = qs[t * sd + d] * before; /* what meets the starting state */
            }
            for (int s = 0; s < i0; s++) k[s * sd + d] *= f;
            done[d] = before * f;
        }
        __syncthreads();
    }
    if (tid < C) ss[tid] = 0.f;
    __syncthreads();
    const float *state = a.states + ((size_t)chunk * a.heads + h) * D * V;
    const int tx = tid & 15, ty = tid >> 4, t4 = ty * 4;
    const bool row_live = t4 < C;
    for (int v0 = 0; v0 < V; v0 += 64) {
        float acc[4][4] = {};
        for (int k0 = 0; k0 < D; k0 += 16) { /* the starting state's part, 16 key channels at a time */
            for (int i = tid; i < 16 * C; i += CHUNK_THREADS) lt[(i & 15) * sc + (i >> 4)] = q[(i >> 4) * sd + k0 + (i & 15)];
            for (int i = tid; i < 16 * 64; i += CHUNK_THREADS)
                rt[i] = v0 + (i & 63) < V ? state[(size_t)(k0 + (i >> 6)) * V + v0 + (i & 63)] : 0.f;
            __syncthreads();
            if (row_live) tile_fma(acc, lt + t4, sc, rt + tx * 4, 64, 16);
            __syncthreads();
        }
        for (int s0 = 0; s0 < n; s0 += 16) { /* the chunk's own part, 16 tokens at a time */
            for (int i = tid; i < 16 * 64; i += CHUNK_THREADS) {
                const int s = s0 + (i >> 6), v = v0 + (i & 63);
                rt[i] = s < n && v < V ? to_f(proj[(size_t)(first + s) * a.ldp + a.off_v + h * V + v]) : 0.f;
            }
            __syncthreads();
            if (row_live) tile_fma(acc, at + s0 * sc + t4, sc, rt + tx * 4, 64, 16);
            __syncthreads();
        }
#pragma unroll
        for (int i = 0; i < 4; i++) {
            float sq = acc[i][0] * acc[i][0] + acc[i][1] * acc[i][1] + acc[i][2] * acc[i][2] + acc[i][3] * acc[i][3];
            for (int o = 8; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o); /* the 16 threads of this token */
            const int t = t4 + i;
            if (t < n) {
                if (tx == 0) ss[t] += sq;
                if (v0 + tx * 4 < V)
                    *reinterpret_cast<float4 *>(a.raw + ((size_t)(first + t) * a.heads + h) * V + v0 + tx * 4) =
                        make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
            }
        }
    }
    __syncthreads(); /* this block's raw outputs and sums are visible to all of its threads */
    for (int i = tid; i < n * V; i += CHUNK_THREADS) {
        const int t = i / V, v = i % V;
        const float rstd = 1.f / sqrtf(ss[t] / (float)a.norm_count + a.eps);
        const float gate = silu(to_f(proj[(size_t)(first + t) * a.ldp + a.off_g + h * V + v]));
        ((T *)a.out)[(size_t)(first + t) * a.ldo + h * V + v] =
            from_f<T>(a.raw[((size_t)(first + t) * a.heads + h) * V + v] * rstd * a.norm[v] * gate);
    }
}

/* ---- chunked form on the tensor cores (bf16 projections, dim <= 256) ------------------------------------------------------ */

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
__device__ __forceinline__ void cp_async16(uint32_t dst, const void *src, bool on) { /* 16 bytes, zeros when off */
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(on ? 16 : 0) : "memory");
}
constexpr int VT = 256; /* columns of v a block handles at a time */

/* The chunk's v rows, columns v0 .. v0 + VT, as bf16 [C][VT + 8]; rows past n and columns past V are zero. */
template <int C, int THREADS = CHUNK_THREADS> __device__ __forceinline__ void stage_v(const ncb_gla &a, uint32_t dst, int first, int n, int h, int v0) {
    const bf16 *v = (const bf16 *)a.proj + (size_t)first * a.ldp + a.off_v + h * a.vdim;
    for (int i = threadIdx.x; i < C * (VT / 8); i += THREADS) {
        const int t = i / (VT / 8), c = v0 + i % (VT / 8) * 8;
        const bool on = t < n && c < a.vdim;
        cp_async16(dst + (t * (VT + 8) + i % (VT / 8) * 8) * 2, v + (on ? (size_t)t * a.ldp + c : 0), on);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
}

/* k_gla_chunk_state with the decayed k as three bf16 terms (24 bits, v is exact): U [dim][vdim] = sum over tokens, dim as M.
 * Grid (chunks, heads, ceil(vdim / VT)). C = 64 for dim <= 128, 32 for dim <= 256: C dim / 256 <= 32 values per thread. */
template <int C> __host__ __device__ inline size_t state_mma_bytes(int D) {
    const size_t work = (size_t)C * D * 4 + (size_t)C * D * 2, terms = (size_t)3 * C * (D + 8) * 2;
    return (size_t)C * (VT + 8) * 2 + (work > terms ? work : terms) + (size_t)2 * D * 4;
}
template <int C> __global__ void __launch_bounds__(CHUNK_THREADS) k_gla_chunk_state_mma(const ncb_gla a) {
    extern __shared__ __align__(16) uint8_t raw[];
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const int chunk = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * VT, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int first = a.chunk_first[chunk], n = a.chunk_count[chunk], D = a.dim, V = a.vdim, HD = a.heads * D;
    constexpr int HALF = C / 2;
    bf16 *vs = reinterpret_cast<bf16 *>(raw);
    uint8_t *rest = raw + C * (VT + 8) * 2;
    float *al = reinterpret_cast<float *>(rest);           /* [C][D], then the terms of k over it */
    bf16 *ks = reinterpret_cast<bf16 *>(al + C * D);       /* [C][D] */
    bf16 *terms = reinterpret_cast<bf16 *>(rest);          /* [3][C][D + 8] */
    const size_t work = (size_t)C * D * 6, three = (size_t)3 * C * (D + 8) * 2;
    float *total = reinterpret_cast<float *>(rest + (work > three ? work : three)); /* [2][D]: the halves' products */
    stage_v<C>(a, smem_addr(vs), first, n, h, v0);
    for (int i = tid; i < C * (D / 4); i += CHUNK_THREADS) {
        const int t = i / (D / 4), d = i % (D / 4) * 4;
        cp_async16(smem_addr(al + t * D + d), a.decay + (size_t)(first + (t < n ? t : 0)) * HD + h * D + d, t < n);
    }
    for (int i = tid; i < C * (D / 8); i += CHUNK_THREADS) {
        const int t = i / (D / 8), d = i % (D / 8) * 8;
        cp_async16(smem_addr(ks + t * D + d), (const bf16 *)a.proj + (size_t)(first + (t < n ? t : 0)) * a.ldp + a.off_k + h * D + d, t < n);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    /* suffix products: item (d, half) walks its half of the tokens backwards */
    float vals[32];
#pragma unroll
    for (int j = 0; j < 32 / HALF; j++) {
        const int item = tid + j * CHUNK_THREADS, d = item % D, half = item / D;
        if (item < 2 * D) {
            float f = 1.f;
#pragma unroll
            for (int i = HALF - 1; i >= 0; i--) {
                const int t = half * HALF + i;
                vals[j * HALF + i] = to_f(ks[t * D + d]) * f;
                if (t < n) f *= al[t * D + d];
            }
            total[half * D + d] = f;
        }
    }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < 32 / HALF; j++) {
        const int item = tid + j * CHUNK_THREADS, d = item % D, half = item / D;
        if (item < 2 * D) {
            const float after = half == 0 ? total[D + d] : 1.f;
#pragma unroll
            for (int i = 0; i < HALF; i++) {
                const float x = vals[j * HALF + i] * after;
                const bf16 hi = __float2bfloat16_rn(x), mid = __float2bfloat16_rn(x - to_f(hi)), lo = __float2bfloat16_rn(x - to_f(hi) - to_f(mid));
                bf16 *p = terms + (half * HALF + i) * (D + 8) + d;
                p[0] = hi, p[C * (D + 8)] = mid, p[2 * C * (D + 8)] = lo;
            }
            if (half == 0 && blockIdx.z == 0) a.chunk_decay[(size_t)chunk * HD + h * D + d] = total[d] * after;
        }
    }
    __syncthreads();
    float *out = a.states + ((size_t)chunk * a.heads + h) * D * V;
    const int g = lane >> 2, t2 = (lane & 3) * 2, col0 = warp * 32;
    if (v0 + col0 >= V) return;
    const uint32_t vb = smem_addr(vs) + ((lane & 15) * (VT + 8) + col0 + (lane >> 4) * 8) * 2;
    const uint32_t kb = smem_addr(terms) + (((lane >> 4) * 8 + (lane & 7)) * (D + 8) + ((lane >> 3) & 1) * 8) * 2;
    for (int m0 = 0; m0 < D; m0 += 32) { /* two 16-row tiles of key channels at a time */
        float acc[2][4][4];
#pragma unroll
        for (int i = 0; i < 32; i++) acc[i >> 4][(i >> 2) & 3][i & 3] = 0.f;
        const int mts = D - m0 >= 32 ? 2 : 1;
#pragma unroll
        for (int k = 0; k < C / 16; k++) {
            uint32_t b[2][4];
            ldsm4_t(b[0], vb + k * 16 * (VT + 8) * 2);
            ldsm4_t(b[1], vb + k * 16 * (VT + 8) * 2 + 32);
#pragma unroll
            for (int m = 0; m < 2; m++)
                if (m < mts) {
#pragma unroll
                    for (int e = 0; e < 3; e++) {
                        uint32_t x[4];
                        ldsm4_t(x, kb + ((e * C + k * 16) * (D + 8) + m0 + m * 16) * 2);
#pragma unroll
                        for (int c = 0; c < 4; c++) mma_bf16(acc[m][c], x, b[c >> 1][(c & 1) * 2], b[c >> 1][(c & 1) * 2 + 1]);
                    }
                }
        }
#pragma unroll
        for (int m = 0; m < 2; m++)
#pragma unroll
            for (int c = 0; c < 4; c++) {
                const int v = v0 + col0 + c * 8 + t2, d = m0 + m * 16 + g;
                if (m < mts && v < V) {
                    *reinterpret_cast<float2 *>(out + (size_t)d * V + v) = make_float2(acc[m][c][0], acc[m][c][1]);
                    *reinterpret_cast<float2 *>(out + (size_t)(d + 8) * V + v) = make_float2(acc[m][c][2], acc[m][c][3]);
                }
            }
    }
}

/* k_gla_chunk_out on the tensor cores, sub-chunks side by side. Per sub-chunk i of 16 tokens: q with the decays since its start
 * (qs), k with the decays to its end (kd), its whole product G_i; all kept as two bf16 terms. Then
 *   scores inside a sub-chunk: a warp per (sub-chunk, four s), products running along t in fp32, lanes over key channels;
 *   scores against sub-chunk j < i: a warp per pair, (qs_i G_(j+1) .. G_(i-1)) . kd_j, three MMAs per step (two-term operands);
 *   output: (qs_i G_0 .. G_(i-1)) S with S as two terms, plus scores (two terms) times v; a warp per 16 columns.
 * Grid (chunks, heads), C = 16 MT, 512 threads. */
constexpr int OUT_THREADS = 512, OUT_WARPS = OUT_THREADS / 32;
template <int MT> __host__ __device__ inline size_t out_mma_bytes(int D) {
    constexpr int C = 16 * MT;
    return (size_t)C * (VT + 8) * 2 + (size_t)2 * C * (C + 8) * 2 + (size_t)4 * C * (D + 8) * 2 /* v, scores, qs, kd */
           + (size_t)2 * C * D * 2 + ((size_t)C * D + MT * D + OUT_WARPS * C + C) * 4;          /* q, k, alpha, G, sums, rstd */
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
/* The two-term pair (hi, lo) times f0, f1 as a new two-term pair. */
__device__ __forceinline__ void rescale2(uint32_t &hi, uint32_t &lo, float f0, float f1) {
    const float2 h = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&hi)), l = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&lo));
    split2((h.x + l.x) * f0, (h.y + l.y) * f1, hi, lo);
}
template <int MT> __global__ void __launch_bounds__(OUT_THREADS, 1) k_gla_chunk_out_mma(const ncb_gla a) {
    extern __shared__ __align__(16) uint8_t raw[];
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    constexpr int C = 16 * MT, sc = C + 8;
    const int chunk = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int first = a.chunk_first[chunk], n = a.chunk_count[chunk], D = a.dim, V = a.vdim, HD = a.heads * D, sq = D + 8;
    bf16 *vs = reinterpret_cast<bf16 *>(raw);                     /* [C][VT + 8] */
    bf16 *at = vs + C * (VT + 8);                                 /* [2][C][sc]: scores' terms, [t][s] */
    bf16 *qs = at + 2 * C * sc, *kd = qs + 2 * C * sq;            /* [2][C][sq] each */
    bf16 *q = kd + 2 * C * sq, *k = q + C * D;                    /* [C][D], as projected */
    float *al = reinterpret_cast<float *>(k + C * D), *G = al + C * D, *sums = G + MT * D, *rstd = sums + OUT_WARPS * C;
    const bf16 *proj = (const bf16 *)a.proj;
    for (int i = tid; i < C * (D / 4); i += OUT_THREADS) {
        const int t = i / (D / 4), d = i % (D / 4) * 4;
        cp_async16(smem_addr(al + t * D + d), a.decay + (size_t)(first + (t < n ? t : 0)) * HD + h * D + d, t < n);
    }
    for (int i = tid; i < C * (D / 8); i += OUT_THREADS) {
        const int t = i / (D / 8), d = i % (D / 8) * 8;
        const bf16 *p = proj + (size_t)(first + (t < n ? t : 0)) * a.ldp + h * D + d;
        cp_async16(smem_addr(q + t * D + d), p + a.off_q, t < n);
        cp_async16(smem_addr(k + t * D + d), p + a.off_k, t < n);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    stage_v<C, OUT_THREADS>(a, smem_addr(vs), first, n, h, 0);
    for (int i = tid; i < C * sc; i += OUT_THREADS) reinterpret_cast<uint32_t *>(at)[i] = 0u; /* both terms */
    for (int i = tid; i < OUT_WARPS * C; i += OUT_THREADS) sums[i] = 0.f;
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    for (int i = tid; i < MT * D; i += OUT_THREADS) { /* alpha, q and k of tokens past n are zero */
        const int sub = i / D, d = i - sub * D;
        float f = 1.f, v[SUB];
#pragma unroll
        for (int t = 0; t < SUB; t++) {
            v[t] = al[(sub * SUB + t) * D + d];
            f *= v[t];
            const int r = sub * SUB + t;
            const float x = to_f(q[r * D + d]) * a.q_scale * f;
            const bf16 hi = __float2bfloat16_rn(x);
            qs[r * sq + d] = hi;
            qs[(C + r) * sq + d] = __float2bfloat16_rn(x - to_f(hi));
        }
        G[i] = f;
        f = 1.f;
#pragma unroll
        for (int t = SUB - 1; t >= 0; t--) {
            const int r = sub * SUB + t;
            const float x = to_f(k[r * D + d]) * f;
            const bf16 hi = __float2bfloat16_rn(x);
            kd[r * sq + d] = hi;
            kd[(C + r) * sq + d] = __float2bfloat16_rn(x - to_f(hi));
            f *= v[t];
        }
    }
    __syncthreads();
    const int g = lane >> 2, t2 = (lane & 3) * 2;
    auto put_score = [&](int t, int s, float v) {
        const bf16 hi = __float2bfloat16_rn(v);
        at[t * sc + s] = hi;
        at[(C + t) * sc + s] = __float2bfloat16_rn(v - to_f(hi));
    };
    for (int task = warp; task < MT * (MT - 1) / 2; task += OUT_WARPS) { /* pairs (i, j), j < i */
        int i = 1, j = task;
        while (j >= i) j -= i, i++;
        if (i * SUB >= n) continue;
        float acc[2][4] = {};
        const uint32_t xa = smem_addr(qs) + ((i * SUB + (lane & 15)) * sq + (lane >> 4) * 8) * 2;
        const uint32_t ya = smem_addr(kd) + ((j * SUB + (lane >> 4) * 8 + (lane & 7)) * sq + ((lane >> 3) & 1) * 8) * 2;
        for (int d0 = 0; d0 < D; d0 += 16) {
            uint32_t xh[4], xl[4], yh[4], yl[4];
            ldsm4(xh, xa + d0 * 2);
            ldsm4(xl, xa + (C * sq + d0) * 2);
            ldsm4(yh, ya + d0 * 2);
            ldsm4(yl, ya + (C * sq + d0) * 2);
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
            for (int e = 0; e < 4; e++) put_score(i * SUB + g + (e >> 1) * 8, j * SUB + c * 8 + t2 + (e & 1), acc[c][e]);
    }
    for (int task = OUT_WARPS - 1 - warp; task < MT * 4; task += OUT_WARPS) { /* (sub-chunk, four s) */
        const int i0 = task / 4 * SUB, s0 = task % 4 * 4;
        if (i0 >= n) continue;
        float acc[64]; /* [s][t] */
#pragma unroll
        for (int e = 0; e < 64; e++) acc[e] = 0.f;
        for (int d = lane; d < D; d += 32) {
            float f[4];
#pragma unroll
            for (int e = 0; e < 4; e++) f[e] = to_f(k[(i0 + s0 + e) * D + d]) * a.q_scale;
#pragma unroll
            for (int t = 0; t < SUB; t++) {
                if (t < s0) continue;
                const float x = to_f(q[(i0 + t) * D + d]), al_t = al[(i0 + t) * D + d];
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    if (t > s0 + e) f[e] *= al_t;
                    if (t >= s0 + e) acc[e * 16 + t] = fmaf(x, f[e], acc[e * 16 + t]);
                }
            }
        }
        reduce64(acc, lane);
        const int at0 = 2 * lane;
#pragma unroll
        for (int e = 0; e < 2; e++) {
            const int s = s0 + (at0 + e) / 16, t = (at0 + e) % 16;
            if (t >= s) put_score(i0 + t, i0 + s, acc[e]);
        }
    }
    __syncthreads();
    for (int i = tid; i < (MT - 1) * D / 2; i += OUT_THREADS) { /* qs <- qs G_0 .. G_(sub - 1), channels d, d + 1 */
        const int sub = 1 + i / (D / 2), d = i % (D / 2) * 2;
        float f0 = 1.f, f1 = 1.f;
        for (int m = 0; m < sub; m++) f0 *= G[m * D + d], f1 *= G[m * D + d + 1];
#pragma unroll 4
        for (int t = 0; t < SUB; t++) {
            uint32_t *hi = reinterpret_cast<uint32_t *>(qs + (sub * SUB + t) * sq + d), *lo = reinterpret_cast<uint32_t *>(qs + (C + sub * SUB + t) * sq + d);
            uint32_t x = *hi, y = *lo;
            rescale2(x, y, f0, f1);
            *hi = x, *lo = y;
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    const float *state = a.states + ((size_t)chunk * a.heads + h) * D * V;
    const int col0 = warp * 16;
    const uint32_t qb = smem_addr(qs) + ((lane & 15) * sq + (lane >> 4) * 8) * 2, ab = smem_addr(at) + ((lane & 15) * sc + (lane >> 4) * 8) * 2;
    const uint32_t vb = smem_addr(vs) + ((lane & 15) * (VT + 8) + col0 + (lane >> 4) * 8) * 2;
    const bool direct = V <= VT; /* the whole row of a token is in this block's registers */
    for (int v0 = 0; v0 < V; v0 += VT) {
        if (v0 > 0) {
            __syncthreads();
            stage_v<C, OUT_THREADS>(a, smem_addr(vs), first, n, h, v0);
            asm volatile("cp.async.wait_group 0;" ::: "memory");
            __syncthreads();
        }
        float acc[MT][2][4];
#pragma unroll
        for (int i = 0; i < MT * 8; i++) acc[i >> 3][(i >> 2) & 1][i & 3] = 0.f;
        const bool live = v0 + col0 < V; /* vdim is a multiple of 16: both column tiles or none */
        constexpr int DEPTH = 3;         /* k-steps of the state in flight */
        float next[DEPTH][2][4];
        auto load = [&](int k0, int slot) {
#pragma unroll
            for (int c = 0; c < 2; c++) {
                const float *p = state + (size_t)(k0 + t2) * V + v0 + col0 + c * 8 + g;
                const bool on = live && k0 < D;
                next[slot][c][0] = on ? p[0] : 0.f, next[slot][c][1] = on ? p[V] : 0.f;
                next[slot][c][2] = on ? p[(size_t)8 * V] : 0.f, next[slot][c][3] = on ? p[(size_t)9 * V] : 0.f;
            }
        };
#pragma unroll
        for (int j = 0; j < DEPTH; j++) load(16 * j, j);
        for (int kb = 0; kb < D; kb += 16 * DEPTH) {
#pragma unroll
            for (int j = 0; j < DEPTH; j++) {
                const int k0 = kb + 16 * j;
                if (k0 >= D) break;
                uint32_t hi[2][2], lo[2][2];
#pragma unroll
                for (int c = 0; c < 2; c++) split2(next[j][c][0], next[j][c][1], hi[c][0], lo[c][0]), split2(next[j][c][2], next[j][c][3], hi[c][1], lo[c][1]);
                load(k0 + 16 * DEPTH, j);
#pragma unroll
                for (int m = 0; m < MT; m++) {
                    uint32_t xh[4], xl[4];
                    ldsm4(xh, qb + (m * 16 * sq + k0) * 2);
                    ldsm4(xl, qb + ((C + m * 16) * sq + k0) * 2);
#pragma unroll
                    for (int c = 0; c < 2; c++) {
                        mma_bf16(acc[m][c], xh, hi[c][0], hi[c][1]);
                        mma_bf16(acc[m][c], xh, lo[c][0], lo[c][1]);
                        mma_bf16(acc[m][c], xl, hi[c][0], hi[c][1]);
                    }
                }
            }
        }
#pragma unroll
        for (int kk = 0; kk < MT; kk++) { /* 16 tokens of the chunk itself; rows before them see none of it */
            uint32_t b[4];
            ldsm4_t(b, vb + kk * 16 * (VT + 8) * 2);
#pragma unroll
            for (int m = kk; m < MT; m++) {
                uint32_t xh[4], xl[4];
                ldsm4(xh, ab + (m * 16 * sc + kk * 16) * 2);
                ldsm4(xl, ab + ((C + m * 16) * sc + kk * 16) * 2);
#pragma unroll
                for (int c = 0; c < 2; c++) {
                    mma_bf16(acc[m][c], xh, b[2 * c], b[2 * c + 1]);
                    mma_bf16(acc[m][c], xl, b[2 * c], b[2 * c + 1]);
                }
            }
        }
#pragma unroll
        for (int m = 0; m < MT; m++)
#pragma unroll
            for (int r = 0; r < 2; r++) {
                float s = 0.f;
#pragma unroll
                for (int c = 0; c < 2; c++) s += acc[m][c][2 * r] * acc[m][c][2 * r] + acc[m][c][2 * r + 1] * acc[m][c][2 * r + 1];
                s += __shfl_xor_sync(0xffffffffu, s, 1);
                s += __shfl_xor_sync(0xffffffffu, s, 2);
                if ((lane & 3) == 0) sums[warp * C + m * 16 + r * 8 + g] += s;
            }
        if (direct) {
            __syncthreads();
            if (tid < C) {
                float s = 0.f;
                for (int w = 0; w < OUT_WARPS; w++) s += sums[w * C + tid];
                rstd[tid] = 1.f / sqrtf(s / (float)a.norm_count + a.eps);
            }
            __syncthreads();
        }
        if (!live) continue;
#pragma unroll
        for (int m = 0; m < MT; m++)
#pragma unroll
            for (int r = 0; r < 2; r++) {
                const int t = m * 16 + r * 8 + g;
                if (t >= n) continue;
                const bf16 *gp = proj + (size_t)(first + t) * a.ldp + a.off_g + h * V;
#pragma unroll
                for (int c = 0; c < 2; c++) {
                    const int v = v0 + col0 + c * 8 + t2;
                    if (direct) {
                        const float2 z = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(gp + v));
                        const float2 w = *reinterpret_cast<const float2 *>(a.norm + v);
                        *reinterpret_cast<__nv_bfloat162 *>((bf16 *)a.out + (size_t)(first + t) * a.ldo + h * V + v) =
                            __floats2bfloat162_rn(acc[m][c][2 * r] * rstd[t] * w.x * silu(z.x), acc[m][c][2 * r + 1] * rstd[t] * w.y * silu(z.y));
                    } else {
                        *reinterpret_cast<float2 *>(a.raw + ((size_t)(first + t) * a.heads + h) * V + v) =
                            make_float2(acc[m][c][2 * r], acc[m][c][2 * r + 1]);
                    }
                }
            }
    }
    if (direct) return;
    __syncthreads();
    if (tid < C) {
        float s = 0.f;
        for (int w = 0; w < OUT_WARPS; w++) s += sums[w * C + tid];
        rstd[tid] = 1.f / sqrtf(s / (float)a.norm_count + a.eps);
    }
    __syncthreads(); /* this block's raw outputs are visible to all of its threads */
    for (int i = tid; i < n * V; i += OUT_THREADS) {
        const int t = i / V, v = i % V;
        const float gate = silu(to_f(proj[(size_t)(first + t) * a.ldp + a.off_g + h * V + v]));
        ((bf16 *)a.out)[(size_t)(first + t) * a.ldo + h * V + v] =
            __float2bfloat16_rn(a.raw[((size_t)(first + t) * a.heads + h) * V + v] * rstd[t] * a.norm[v] * gate);
    }
}

/* ---- host side ------------------------------------------------------------------------------------------------------ */

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

int check(const ncb_gla &g) {
    if (g.rows < 0 || g.rows > 0x7fffff00LL || g.heads <= 0 || g.heads > 65535 || g.dim <= 0 || g.vdim <= 0 || g.dim % 16 ||
        g.vdim % 16 || g.rank <= 0 || g.norm_count <= 0 || g.n_slots <= 0)
        return NCB_ERR_ARG;
    if (g.rows == 0) return NCB_OK;
    if (!g.proj || !g.a2 || !g.a2_bias || !g.norm || !g.state || !g.pos) return NCB_ERR_ARG;
    return ((uintptr_t)g.state | (uintptr_t)g.states | (uintptr_t)g.raw) % 16 ? NCB_ERR_ALIGN : NCB_OK;
}

size_t step_smem(const ncb_gla &g, int slices) {
    const int VS = g.vdim / slices, dgs = STEP_THREADS / (VS / 4);
    return (3 * (size_t)g.dim + (size_t)dgs * VS + VS + STEP_THREADS / 32) * sizeof(float);
}

} /* namespace */

extern "C" {

/* Tokens per chunk of the chunked form for key size `dim`; 0: only the token-by-token form takes it. */
int gla_chunk_tokens(int dim) { return dim <= 0 ? 0 : dim <= 128 ? 64 : dim <= 256 ? 32 : dim <= 512 ? 16 : 0; }

int gla_step(const ncb_gla *g, int f32, void *stream) {
    if (!g) return NCB_ERR_ARG;
    const int rc = check(*g);
    if (rc != NCB_OK || g->rows == 0) return rc;
    const int segments = g->seg_first ? g->n_segments : (int)g->rows;
    if (segments <= 0 || segments > 65535 || (g->seg_first && !g->seg_count)) return NCB_ERR_ARG;
    /* vdim slices: enough blocks for the GPU, slices of at least 16 values and at most what the threads cover */
    int slices = 1;
    while (slices < 8 && g->vdim % (2 * slices * 16) == 0 &&
           (g->vdim / slices > 4 * STEP_THREADS || (long long)segments * g->heads * slices < 148))
        slices *= 2;
    if (g->vdim / slices > 4 * STEP_THREADS) return NCB_ERR_UNSUPPORTED;
    const size_t smem = step_smem(*g, slices);
    if (smem > 200 * 1024) return NCB_ERR_UNSUPPORTED;
    const dim3 grid(slices, g->heads, segments);
    return f32 ? launch(k_gla_step<float>, grid, STEP_THREADS, smem, slices, (cudaStream_t)stream, *g)
               : launch(k_gla_step<bf16>, grid, STEP_THREADS, smem, slices, (cudaStream_t)stream, *g);
}

int gla_chunked(const ncb_gla *g, int f32, void *stream_ptr) {
    if (!g) return NCB_ERR_ARG;
    int rc = check(*g);
    if (rc != NCB_OK || g->rows == 0) return rc;
    const int C = gla_chunk_tokens(g->dim);
    if (C == 0 || C != g->chunk) return NCB_ERR_UNSUPPORTED;
    if (g->n_chunks <= 0 || g->n_segments <= 0 || g->n_segments > 65535 || !g->seg_first || !g->seg_chunk || !g->chunk_first ||
        !g->chunk_count || !g->decay || !g->chunk_decay || !g->states || (g->out && !g->raw))
        return NCB_ERR_ARG;
    cudaStream_t stream = (cudaStream_t)stream_ptr;
    const size_t decay_smem = (size_t)DECAY_ROWS * g->rank * 4, state_smem = ((size_t)C * ((g->dim + 63) / 64 * 64) + (size_t)C * 64) * 4,
                 out_smem = out_floats(C, g->dim) * 4;
    if (decay_smem > 200 * 1024 || out_smem > 226 * 1024) return NCB_ERR_UNSUPPORTED;
    const dim3 decay_grid((unsigned)((g->rows + DECAY_ROWS - 1) / DECAY_ROWS), (g->heads * g->dim + CHUNK_THREADS - 1) / CHUNK_THREADS), state_grid(g->n_chunks, g->heads, (g->vdim + 63) / 64),
        out_grid(g->n_chunks, g->heads),
        scan_grid((unsigned)(((size_t)g->heads * g->dim * g->vdim / 4 + CHUNK_THREADS - 1) / CHUNK_THREADS), g->n_segments);
    rc = f32 ? launch(k_gla_decay<float>, decay_grid, CHUNK_THREADS, decay_smem, 1, stream, *g)
             : launch(k_gla_decay<bf16>, decay_grid, CHUNK_THREADS, decay_smem, 1, stream, *g);
    if (rc != NCB_OK) return rc;
    /* 16-byte copies of rows: every offset of the projection a multiple of 8 */
    const bool mma = !f32 && g->dim <= 256 && !(g->ldp % 8 | g->off_q % 8 | g->off_k % 8 | g->off_v % 8 | g->off_g % 8 | g->ldo % 2) &&
                     !((uintptr_t)g->proj % 16 | (uintptr_t)g->decay % 16);
    if (mma) {
        const dim3 grid(g->n_chunks, g->heads, (g->vdim + VT - 1) / VT);
        rc = C == 64 ? launch(k_gla_chunk_state_mma<64>, grid, CHUNK_THREADS, state_mma_bytes<64>(g->dim), 1, stream, *g)
                     : launch(k_gla_chunk_state_mma<32>, grid, CHUNK_THREADS, state_mma_bytes<32>(g->dim), 1, stream, *g);
        if (rc != NCB_OK) return rc;
        rc = launch(k_gla_scan, scan_grid, CHUNK_THREADS, 0, 1, stream, *g);
        if (rc != NCB_OK || !g->out) return rc;
        return C == 64 ? launch(k_gla_chunk_out_mma<4>, out_grid, OUT_THREADS, out_mma_bytes<4>(g->dim), 1, stream, *g)
                       : launch(k_gla_chunk_out_mma<2>, out_grid, OUT_THREADS, out_mma_bytes<2>(g->dim), 1, stream, *g);
    }
    rc = f32 ? launch(k_gla_chunk_state<float>, state_grid, CHUNK_THREADS, state_smem, 1, stream, *g)
             : launch(k_gla_chunk_state<bf16>, state_grid, CHUNK_THREADS, state_smem, 1, stream, *g);
    if (rc != NCB_OK) return rc;
    rc = launch(k_gla_scan, scan_grid, CHUNK_THREADS, 0, 1, stream, *g);
    if (rc != NCB_OK || !g->out) return rc;
    return f32 ? launch(k_gla_chunk_out<float>, out_grid, CHUNK_THREADS, out_smem, 1, stream, *g)
               : launch(k_gla_chunk_out<bf16>, out_grid, CHUNK_THREADS, out_smem, 1, stream, *g);
}

} /* extern "C" */
