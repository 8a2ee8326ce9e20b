// A short causal convolution over time, channel by channel, on rows that one product has just written:
//   y_t[c] = sum_j w[c][j] u_(t - taps + 1 + j)[c],   zeros before a sequence's first token,
// where u is a column of the step's rows (a bias added, if there is one) and the inputs before the step's first row of a
// sequence come from the slot's kept inputs [taps - 1][C] (row j: taps - 1 - j tokens back, bias included).
#pragma once
#include "common.cuh"

namespace hos {

constexpr int kMaxTaps = 16;

// Channel `ch` (of the C kept ones) of row n, whose sequence's first row of this step is r0; `raw` points at the channel's
// column.  keep_w (only where every sequence of the step brings one token): the kept inputs move on by one here; they are
// the same memory as `keep`, and a channel is one thread's business alone.
__device__ __forceinline__ float short_conv(const float* raw, long long ld, float bias, const float* __restrict__ w, int taps,
                                            const float* keep, float* keep_w, int C, int ch, int n, int r0, bool fresh) {
    float acc = 0.f;
    for (int j = 0; j < taps; ++j) {
        const int src = n - (taps - 1) + j;              // the row of this step that holds the input, if it is one
        float x = 0.f;
        if (src >= r0) x = raw[(size_t)src * ld] + bias;
        else if (!fresh) x = keep[(size_t)((taps - 1) + (src - r0)) * C + ch];
        acc = fmaf(w[(size_t)ch * taps + j], x, acc);
        if (keep_w != nullptr && j >= 1) keep_w[(size_t)(j - 1) * C + ch] = x;      // row j - 1 is read before this
    }
    return acc;
}

// The last taps - 1 inputs of every sequence of the step go to the slot's kept inputs: a thread per (sequence, channel).
// raw: the rows from the first channel's column on; bias: [C] or null.
static __global__ void short_conv_keep_kernel(const float* __restrict__ raw, long long ld, const float* __restrict__ bias, int taps,
                                              float* __restrict__ conv_state, const int* __restrict__ token_pos,
                                              const int* __restrict__ token_seq, const int* __restrict__ cu_seqlens,
                                              const int* __restrict__ seq_slot, int C) {
    pdl_enter();
    const int seq = blockIdx.y;
    const int ch = blockIdx.x * blockDim.x + threadIdx.x;
    const int r0 = cu_seqlens[seq], r1 = cu_seqlens[seq + 1];
    if (ch >= C || r1 <= r0 || token_seq[r0] < 0) return;
    const bool fresh = token_pos[r0] == 0;
    const float b = bias != nullptr ? bias[ch] : 0.f;
    float* keep = conv_state + (size_t)seq_slot[seq] * (taps - 1) * C;
    float nv[kMaxTaps];
#pragma unroll
    for (int j = 0; j < kMaxTaps; ++j) {
        if (j < taps - 1) {
            const int src = r1 - (taps - 1) + j;
            nv[j] = src >= r0 ? raw[(size_t)src * ld + ch] + b : (fresh ? 0.f : keep[(size_t)((taps - 1) + (src - r0)) * C + ch]);
        }
    }
#pragma unroll
    for (int j = 0; j < kMaxTaps; ++j)
        if (j < taps - 1) keep[(size_t)j * C + ch] = nv[j];
}

}  // namespace hos
