/*
 * The state a short convolution carries from pass to pass: the last taps - 1 projected rows of every sequence go into its
 * ring (short_conv.cuh) once everything that reads the ring has run. The convolution itself is part of the mixers' kernels.
 */
#include "short_conv.cuh"

namespace {

constexpr int THREADS = 128;

/* One block per row; only a sequence's last rows in the pass have something to do. */
template <typename T> __global__ void __launch_bounds__(THREADS) k_conv_tail(const ncb_conv c, int *status) {
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const int row = blockIdx.x, pos = c.pos[row], slot = c.slot_map ? c.slot_map[row] : row, later = row + c.taps - 1;
    if (pos < 0) return;
    if (slot < 0 || slot >= c.n_slots) {
        if (threadIdx.x == 0) flag(status, NCB_DEV_BAD_POSITION);
        return;
    }
    if (later < c.rows && c.pos[later] == pos + c.taps - 1 && (c.slot_map ? c.slot_map[later] : later) == slot) return;
    const Place at = {pos, slot, 0};
    for (int ch = 2 * threadIdx.x; ch < c.width; ch += 2 * THREADS) keep2<T>(c, row, at, ch);
}

} /* namespace */

extern "C" int short_conv_tail(const ncb_conv *c, int f32, int *status, void *stream) {
    if (!c) return NCB_ERR_ARG;
    const int rc = check_conv(*c);
    if (rc != NCB_OK || c->rows == 0 || c->taps == 1) return rc;
    const dim3 grid((unsigned)c->rows);
    return f32 ? launch(k_conv_tail<float>, grid, THREADS, 0, 1, (cudaStream_t)stream, *c, status)
               : launch(k_conv_tail<bf16>, grid, THREADS, 0, 1, (cudaStream_t)stream, *c, status);
}
