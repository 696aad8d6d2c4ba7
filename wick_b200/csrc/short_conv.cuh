// A short causal convolution over time, a filter per channel, for steps of any shape: the inputs of earlier steps come
// from the sequence's record (float32, [taps - 1][channels] inputs, oldest first, at its start), which the second kernel
// brings up to date; before position 0 there are zeros.  The sums run over the taps in order.
#pragma once

#include "common.cuh"

namespace wick {

constexpr int CONV_MAX_TAPS = 16;
__device__ __forceinline__ float silu_f(float v) { return v / (1.0f + expf(-v)); }

__device__ __forceinline__ float sum_parts(const float* __restrict__ parts, int splits, int64_t split_stride, int64_t at) {
    float v = 0.f;
    for (int s = 0; s < splits; ++s) v += parts[s * split_stride + at];
    return v;
}

constexpr int CONV_TOKENS = 4;              // tokens a thread of the convolution takes (their loads are in flight together)

// out[t][c] = silu(bias_c + sum over k of w[c][k] u_(p - (taps - 1) + k)), u the partial sums' columns from first_col on.
// grid (ceil(tokens / CONV_TOKENS), ceil(channels / 256)).  ONE: the
// projection came as a single set of sums (its loads need no loop and go out together).
template <bool ONE>
__global__ void __launch_bounds__(256)
short_conv_kernel(const float* __restrict__ parts, int splits, int64_t split_stride, int cols, int first_col, int channels, int taps,
                const float* __restrict__ w, const float* __restrict__ bias, const float* __restrict__ state, int64_t record,
                const int* __restrict__ slots, const int* __restrict__ seq_of_token, const int* __restrict__ positions,
                const int* __restrict__ start, float* __restrict__ out, int n) {
    pdl_trigger();
    pdl_wait();
    parts = fresh(parts);
    state = fresh(state);
    const int c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= channels) return;
    const float b0 = bias ? bias[c] : 0.f;
    float acc[CONV_TOKENS];
    int pos[CONV_TOKENS], first[CONV_TOKENS];
    const float* rec[CONV_TOKENS];
#pragma unroll
    for (int j = 0; j < CONV_TOKENS; ++j) {
        const int t = min(blockIdx.x * CONV_TOKENS + j, n - 1), b = seq_of_token[t];
        pos[j] = positions[t];
        first[j] = start[b];
        rec[j] = state + (int64_t)slots[b] * record;
        acc[j] = b0;
    }
#pragma unroll 4
    for (int k = 0; k < taps; ++k) {
        const float wk = w[(int64_t)c * taps + k];
        float u[CONV_TOKENS];
#pragma unroll
        for (int j = 0; j < CONV_TOKENS; ++j) {
            const int t = min(blockIdx.x * CONV_TOKENS + j, n - 1), sp = pos[j] - (taps - 1) + k;
            u[j] = 0.f;
            const int64_t at = (int64_t)(t - (pos[j] - sp)) * cols + first_col + c;
            if (sp >= first[j]) u[j] = ONE ? parts[at] : sum_parts(parts, splits, split_stride, at);
            else if (sp >= 0) u[j] = rec[j][(int64_t)(sp - (first[j] - (taps - 1))) * channels + c];
        }
#pragma unroll
        for (int j = 0; j < CONV_TOKENS; ++j) acc[j] = fmaf(wk, u[j], acc[j]);
    }
#pragma unroll
    for (int j = 0; j < CONV_TOKENS; ++j) {
        const int t = blockIdx.x * CONV_TOKENS + j;
        if (t < n) out[(int64_t)t * channels + c] = silu_f(acc[j]);
    }
}

// grid (sequences, ceil(channels / 256)).  Runs after the convolution has read the old inputs.
static __global__ void __launch_bounds__(256)
short_conv_state_kernel(const float* __restrict__ parts, int splits, int64_t split_stride, int cols, int first_col, int channels,
                      int taps, float* __restrict__ state, int64_t record, const int* __restrict__ slots,
                      const int* __restrict__ cu_seqlens) {
    pdl_trigger();
    pdl_wait();
    parts = fresh(parts);
    state = fresh(state);
    const int b = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= channels) return;
    const int t0 = cu_seqlens[b], q = cu_seqlens[b + 1] - t0;
    if (q <= 0) return;
    float* rec = state + (int64_t)slots[b] * record;
    float keep[CONV_MAX_TAPS];
#pragma unroll
    for (int j = 0; j < CONV_MAX_TAPS; ++j) {
        if (j >= taps - 1) break;
        const int from = j + q;                                          // where the input of new place j lies now
        keep[j] = from >= taps - 1 ? sum_parts(parts, splits, split_stride, (int64_t)(t0 + from - (taps - 1)) * cols + first_col + c)
                                   : rec[(int64_t)from * channels + c];
    }
#pragma unroll
    for (int j = 0; j < CONV_MAX_TAPS; ++j) {
        if (j >= taps - 1) break;
        rec[(int64_t)j * channels + c] = keep[j];
    }
}

}  // namespace wick
