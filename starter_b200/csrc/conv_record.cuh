// The record of a short causal convolution over time: a sequence's last `taps` - 1 inputs, [taps - 1][channels] floats.
#pragma once
#include "common.cuh"

// A sequence's record becomes its last taps - 1 inputs (after a step of several rows).  p: the step's inputs, rows `ld`
// elements apart.  A step of fewer rows than that keeps the later entries of the old record: a thread reads its channel's
// entries before it writes them.
template <class T>
__global__ void conv_record_kernel(const T* __restrict__ p, long long ld, int taps, float* state, long long state_slot, SbBatch batch, int C) {
    pdl_wait();
    const int s = blockIdx.x, first = batch.cu_q[s], n = batch.cu_q[s + 1] - first, keep = taps - 1;
    float* rec = state + (long long)batch.seq_slot[s] * state_slot;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < C; c += gridDim.y * blockDim.x)
        for (int e = 0; e < keep; ++e) {
            const int src = n - keep + e;
            rec[(long long)e * C + c] = src >= 0 ? to_f<T>(p[(long long)(first + src) * ld + c]) : rec[(long long)(e + n) * C + c];
        }
}

static inline void launch_conv_record(int dtype, const void* p, long long ld, int taps, float* state, long long state_slot, SbBatch batch,
                                      int C, cudaStream_t stream) {
    const dim3 grid(batch.n_seqs, batch.n_seqs < 64 ? (C + 127) / 128 : 1);
    if (dtype == SB_F32)
        sb_launch(conv_record_kernel<float>, grid, 128, 0, stream, (const float*)p, ld, taps, state, state_slot, batch, C);
    else
        sb_launch(conv_record_kernel<__nv_bfloat16>, grid, 128, 0, stream, (const __nv_bfloat16*)p, ld, taps, state, state_slot, batch, C);
}
