/*
 * The state a short convolution carries from pass to pass: the last taps - 1 projected rows of every sequence go into its
 * ring (short_conv.cuh) once everything that reads the ring has run. The convolution itself is part of the mixers' kernels.
 */
#include "short_conv.cuh"

namespace {

constexpr int THREADS = 128;

/* A block looks at THREADS rows and 2 THREADS channels; only a sequence's last rows in the pass have something to keep. */
template <typename T> __global__ void __launch_bounds__(THREADS) k_conv_tail(const ncb_conv c, int *status) {
    __shared__ int rows[THREADS], n_rows;
    if (threadIdx.x == 0) n_rows = 0;
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    __syncthreads();
    const long long row = (long long)blockIdx.x * THREADS + threadIdx.x, later = row + c.taps - 1;
    if (row < c.rows && c.pos[row] >= 0) {
        const int pos = c.pos[row], slot = c.slot_map ? c.slot_map[row] : (int)row;
        if (slot < 0 || slot >= c.n_slots) flag(status, NCB_DEV_BAD_POSITION);
        else if (!(later < c.rows && c.pos[later] == pos + c.taps - 1 && (c.slot_map ? c.slot_map[later] : (int)later) == slot))
            rows[atomicAdd(&n_rows, 1)] = (int)row;
    }
    __syncthreads();
    const int ch = 2 * (blockIdx.y * THREADS + threadIdx.x);
    if (ch >= c.width) return;
#pragma unroll 4
    for (int i = 0; i < n_rows; i++) { /* (their places in the rings differ: any order) */
        const int r = rows[i];
        const Place at = {c.pos[r], c.slot_map ? c.slot_map[r] : r, 0};
        keep2<T>(c, r, at, ch);
    }
}

} /* namespace */

extern "C" int short_conv_tail(const ncb_conv *c, int f32, int *status, void *stream) {
    if (!c) return NCB_ERR_ARG;
    const int rc = check_conv(*c);
    if (rc != NCB_OK || c->rows == 0 || c->taps == 1) return rc;
    const dim3 grid((unsigned)((c->rows + THREADS - 1) / THREADS), (c->width + 2 * THREADS - 1) / (2 * THREADS));
    return f32 ? launch(k_conv_tail<float>, grid, THREADS, 0, 1, (cudaStream_t)stream, *c, status)
               : launch(k_conv_tail<bf16>, grid, THREADS, 0, 1, (cudaStream_t)stream, *c, status);
}
