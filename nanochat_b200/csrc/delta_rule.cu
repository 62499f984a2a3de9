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

} /* namespace */

extern "C" {

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
