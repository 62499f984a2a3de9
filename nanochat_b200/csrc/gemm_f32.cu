/*
 * y = epilogue(x . W^T) entirely in fp32 (fused multiply-adds on the CUDA cores, no reduced-precision matrix mode): the
 * GEMMs of a model that runs with 32-bit weights and activations, on the same fp32 residual stream and with the same
 * epilogues as the bf16 GEMM libraries (ncb_gemm_rs). It exists for exactness, not for speed: a plain 64 x 64 tile per
 * block, both operands staged through shared memory 16 k-values at a time, 4 x 4 products per thread.
 */
#include "gemm_rs.cuh"

namespace {

constexpr int TM = 64, TN = 64, TK = 16, THREADS = 256;
enum { EPI_STORE = 0, EPI_F32 = 3, EPI_GEGLU = 5, EPI_STREAM = 6, EPI_STREAMS = 7, EPI_SWIGLU = 8 };

struct Args {
    const float *x, *w;
    float *y;
    long long rows, ldy;
    int N, K, n_store, epilogue;
    StreamIO rs;
};

__global__ void __launch_bounds__(THREADS) k_gemm_f32(const Args a) {
    __shared__ float xs[TK][TM + 4], ws[TK][TN + 4];
    __shared__ float factor[TM];
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const long long m0 = (long long)blockIdx.x * TM;
    const int n0 = blockIdx.y * TN;
    { /* row factors: four threads per row */
        const int r = tid >> 2;
        float s = 0.f;
        if (a.rs.ss && m0 + r < a.rows)
            for (int i = tid & 3; i < a.rs.ss_parts; i += 4) s += a.rs.ss[(m0 + r) * a.rs.ss_parts + i];
        s += __shfl_xor_sync(0xffffffffu, s, 1);
        s += __shfl_xor_sync(0xffffffffu, s, 2);
        if ((tid & 3) == 0) factor[r] = row_scale(a.rs, s);
    }
    float acc[4][4] = {};
    const int lr = tid >> 2, lk = (tid & 3) * 4; /* each thread stages four k-values of one row of x and of W */
    for (int k0 = 0; k0 < a.K; k0 += TK) {
        const float4 xv = m0 + lr < a.rows ? *reinterpret_cast<const float4 *>(a.x + (m0 + lr) * a.K + k0 + lk)
                                           : make_float4(0.f, 0.f, 0.f, 0.f);
        const float4 wv = *reinterpret_cast<const float4 *>(a.w + (size_t)(n0 + lr) * a.K + k0 + lk);
        __syncthreads();
        xs[lk][lr] = xv.x, xs[lk + 1][lr] = xv.y, xs[lk + 2][lr] = xv.z, xs[lk + 3][lr] = xv.w;
        ws[lk][lr] = wv.x, ws[lk + 1][lr] = wv.y, ws[lk + 2][lr] = wv.z, ws[lk + 3][lr] = wv.w;
        __syncthreads();
#pragma unroll
        for (int k = 0; k < TK; k++) {
            float xa[4], wa[4];
#pragma unroll
            for (int i = 0; i < 4; i++) xa[i] = xs[k][ty * 4 + i], wa[i] = ws[k][tx * 4 + i];
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(xa[i], wa[j], acc[i][j]);
        }
    }
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const int r = ty * 4 + i, n = n0 + tx * 4;
        const long long row = m0 + r;
        const bool live = row < a.rows;
        float v[4];
#pragma unroll
        for (int j = 0; j < 4; j++) v[j] = acc[i][j] * factor[r];
        if (a.epilogue == EPI_SWIGLU) {
            if (live) {
                a.y[row * a.ldy + (n >> 1)] = silu(v[0]) * v[1];
                a.y[row * a.ldy + (n >> 1) + 1] = silu(v[2]) * v[3];
            }
        } else if (a.epilogue == EPI_GEGLU) {
            if (live) {
                a.y[row * a.ldy + (n >> 1)] = gelu_tanh(v[0]) * v[1];
                a.y[row * a.ldy + (n >> 1) + 1] = gelu_tanh(v[2]) * v[3];
            }
        } else if (a.epilogue == EPI_STREAM || a.epilogue == EPI_STREAMS) {
            float q = 0.f;
            if (live)
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    const size_t at = (size_t)row * a.N + n + j;
                    const float h = a.epilogue == EPI_STREAM ? stream_add(a.rs, at, v[j]) : streams_add(a.rs, row, n + j, a.N, v[j]);
                    reinterpret_cast<float *>(a.rs.x_next)[at] = h * a.rs.gain[n + j];
                    q += h * h;
                }
            for (int o = 8; o > 0; o >>= 1) q += __shfl_xor_sync(0xffffffffu, q, o); /* the 16 threads of this row */
            if (live && tx == 0) a.rs.ss_next[row * gridDim.y + blockIdx.y] = q;
        } else if (live) {
#pragma unroll
            for (int j = 0; j < 4; j++)
                if (n + j < a.n_store) a.y[row * a.ldy + n + j] = v[j];
        }
    }
}

} /* namespace */

extern "C" int gemm_f32_rs(const ncb_gemm_rs *g, void *stream) {
    if (!g || g->rows > 0x7fffff00LL || g->N % TN || g->K % 64) return NCB_ERR_ARG;
    const int rc = check_rs(*g);
    if (rc != NCB_OK || g->rows == 0) return rc;
    const Args a = {(const float *)g->x, (const float *)g->w, (float *)g->y, g->rows, g->ldy, g->N, g->K, g->n_store,
                    g->epilogue, stream_io(*g)};
    cudaLaunchConfig_t config = {};
    config.gridDim = dim3((unsigned)((g->rows + TM - 1) / TM), g->N / TN);
    config.blockDim = dim3(THREADS);
    config.stream = (cudaStream_t)stream;
    cudaLaunchAttribute attribute[1];
    attribute[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attribute[0].val.programmaticStreamSerializationAllowed = 1;
    config.attrs = attribute;
    config.numAttrs = 1;
    return cudaLaunchKernelEx(&config, k_gemm_f32, a) == cudaSuccess ? NCB_OK : NCB_ERR_LAUNCH;
}
