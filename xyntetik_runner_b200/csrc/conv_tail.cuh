// The tail of a short causal convolution that a request carries from step to step.
#pragma once
#include "common.cuh"

// tail[j] <- the input at place len - (taps - 1) + j of the portion: a row of this step, or, where the portion is
// shorter than the tail, what the tail held len places further on.  All blocks of the scan that walk a portion share
// its channels (block `part` of `parts`), after the kernel that read the old tail is complete; a thread reads all of a
// channel's values before it writes any (eight at a time: the reads of a pass lie ahead of its writes, j ascends).
template <typename T>
__device__ __forceinline__ void xr_tail_update(const T* __restrict__ proj, long long ldp, float* tail, int start, int len,
                                               int CH, int taps, int part, int parts) {
    for (int c = part * blockDim.x + threadIdx.x; c < CH; c += parts * blockDim.x)
        for (int j0 = 0; j0 < taps - 1; j0 += 8) {
            float x[8];
#pragma unroll
            for (int i = 0; i < 8; i++) {
                const int j = j0 + i, src = len - (taps - 1) + j;
                x[i] = j >= taps - 1 ? 0.f : (src >= 0 ? xr_to_f32<T>(proj[(size_t)(start + src) * ldp + c]) : tail[(size_t)(j + len) * CH + c]);
            }
#pragma unroll
            for (int i = 0; i < 8; i++)
                if (j0 + i < taps - 1) tail[(size_t)(j0 + i) * CH + c] = x[i];
        }
}
