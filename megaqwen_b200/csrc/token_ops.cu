// Token-list helpers of the device-resident decode chains (both libraries).
#include <cuda_runtime.h>

#include "../../include/megaqwen_b200.h"

namespace {

__global__ void k_fill_iota(int* dst, int start, int n) {
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) dst[i] = start + i;
}

__global__ void k_find_first_eos(const int* tokens, int n, const int* eos, int n_eos, int* out) {
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    const int t = tokens[i];
    for (int j = 0; j < n_eos; ++j)
        if (t == eos[j]) { atomicMin(out, i); return; }
}

}  // namespace

extern "C" int mq_launch_fill_iota(int* dst, int start, int n, void* stream) {
    if (!dst || n < 0) return MQ_ERR_BAD_ARG;
    if (n == 0) return MQ_OK;
    k_fill_iota<<<(n + 255) / 256, 256, 0, (cudaStream_t)stream>>>(dst, start, n);
    return (int)cudaGetLastError();
}

extern "C" int mq_launch_find_first_eos(const int* tokens, int n, const int* eos_ids, int n_eos, int* out_index, void* stream) {
    if (!tokens || !out_index || n < 0 || n_eos < 0 || (n_eos > 0 && !eos_ids)) return MQ_ERR_BAD_ARG;
    if (n == 0 || n_eos == 0) return MQ_OK;
    k_find_first_eos<<<(n + 255) / 256, 256, 0, (cudaStream_t)stream>>>(tokens, n, eos_ids, n_eos, out_index);
    return (int)cudaGetLastError();
}
