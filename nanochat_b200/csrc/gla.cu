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

/* Grid (slices, heads, segments), cluster (slices, 1, 1); segment z = rows first[z] .. + count[z] - 1 of one slot at
 * ascending positions (first NULL: row z alone). */
template <typename T> __global__ void __launch_bounds__(STEP_THREADS) k_gla_step(const ncb_gla a) {
    extern __shared__ float sm[];
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const int tid = threadIdx.x, h = blockIdx.y, slices = gridDim.x, rank = blockIdx.x;
    const int D = a.dim, V = a.vdim, VS = V / slices, v0 = rank * VS;
    const int groups = VS / 4, dgs = STEP_THREADS / groups;
    float *q = sm, *k = q + D, *alpha = k + D, *part = alpha + D, *o = part + dgs * VS, *sums = o + VS;
    __shared__ float block_sum;
    const int first = a.seg_first ? a.seg_first[blockIdx.z] : blockIdx.z, count = a.seg_first ? a.seg_count[blockIdx.z] : 1;
    cg::cluster_group cluster = cg::this_cluster();
    const int pos0 = a.pos[first], slot = a.slot_map ? a.slot_map[first] : first;
    const bool bad = pos0 >= 0 && (slot < 0 || slot >= a.n_slots);
    if (bad && tid == 0) flag(a.status, NCB_DEV_BAD_POSITION);
    if (pos0 < 0 || bad) { /* an idle row: no state touched, a zero output (every block of the cluster takes this exit) */
        if (a.out)
            for (int i = tid; i < count * VS; i += STEP_THREADS)
                ((T *)a.out)[(size_t)(first + i / VS) * a.ldo + h * V + v0 + i % VS] = from_f<T>(0.f);
        return;
    }
    float *state = a.state + ((size_t)slot * a.heads + h) * D * V;
    const int c = tid % groups, dg = tid / groups;
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
#pragma unroll 4
            for (int d = dg; d < D; d += dgs) {
                float4 *sp = reinterpret_cast<float4 *>(state + (size_t)d * V + v0 + 4 * c);
                float4 s = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *sp;
                const float al = alpha[d], kd = k[d], qd = q[d];
                s.x = fmaf(al, s.x, kd * vx), s.y = fmaf(al, s.y, kd * vy);
                s.z = fmaf(al, s.z, kd * vz), s.w = fmaf(al, s.w, kd * vw);
                *sp = s;
                acc.x = fmaf(qd, s.x, acc.x), acc.y = fmaf(qd, s.y, acc.y);
                acc.z = fmaf(qd, s.z, acc.z), acc.w = fmaf(qd, s.w, acc.w);
            }
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
    rc = f32 ? launch(k_gla_chunk_state<float>, state_grid, CHUNK_THREADS, state_smem, 1, stream, *g)
             : launch(k_gla_chunk_state<bf16>, state_grid, CHUNK_THREADS, state_smem, 1, stream, *g);
    if (rc != NCB_OK) return rc;
    rc = launch(k_gla_scan, scan_grid, CHUNK_THREADS, 0, 1, stream, *g);
    if (rc != NCB_OK || !g->out) return rc;
    return f32 ? launch(k_gla_chunk_out<float>, out_grid, CHUNK_THREADS, out_smem, 1, stream, *g)
               : launch(k_gla_chunk_out<bf16>, out_grid, CHUNK_THREADS, out_smem, 1, stream, *g);
}

} /* extern "C" */
