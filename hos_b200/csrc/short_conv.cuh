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

template <int VEC>
__device__ __forceinline__ void conv_load(const float* p, float (&x)[VEC]) {
    if constexpr (VEC == 4) {
        const float4 t = *(const float4*)p;
        x[0] = t.x; x[1] = t.y; x[2] = t.z; x[3] = t.w;
    } else {
        x[0] = *p;
    }
}
template <int VEC>
__device__ __forceinline__ void conv_store(float* p, const float (&x)[VEC]) {
    if constexpr (VEC == 4) *(float4*)p = make_float4(x[0], x[1], x[2], x[3]);
    else *p = x[0];
}

constexpr int kConvTokens = 16;      // consecutive rows that a thread walks at most

// What a walk needs to know.  w: [taps][C]; in_bias (or null): [C], added to the rows' columns before the convolution;
// keep / keep_w: as in short_conv above, from slot 0 on.
struct ConvWalk {
    const float* raw;
    long long ld;
    const float* w;
    const float* in_bias;
    const float* keep;
    float* keep_w;
    const int* token_pos;
    const int* token_seq;
    const int* cu_seqlens;
    const int* seq_slot;
    int taps, C;
};

// The convolution of VEC channels from ch on, over rows n0 .. n1 - 1, with the inputs in sight in registers, so that a
// column is read once; a sequence's first row, or the walk's, fetches the ones before it from the rows or the slot's kept
// inputs.  emit(n, y) takes every live row's result, pad(n) the padding rows.
template <int TAPS, int VEC, typename Emit, typename Pad>
__device__ __forceinline__ void conv_walk(const ConvWalk& c, int ch, int n0, int n1, Emit emit, Pad pad) {
    const int taps = TAPS > 0 ? TAPS : c.taps;
    constexpr int MAXT = TAPS > 0 ? TAPS : kMaxTaps;
    float wr[MAXT][VEC], win[MAXT][VEC], b[VEC];
#pragma unroll
    for (int v = 0; v < VEC; ++v) b[v] = 0.f;
    if (c.in_bias != nullptr) conv_load<VEC>(c.in_bias + ch, b);
#pragma unroll
    for (int j = 0; j < MAXT; ++j) {
#pragma unroll
        for (int v = 0; v < VEC; ++v) wr[j][v] = win[j][v] = 0.f;
        if (j < taps) conv_load<VEC>(c.w + (size_t)j * c.C + ch, wr[j]);
    }
    int last_seq = -2;
    for (int n = n0; n < n1; ++n) {
        const int seq = c.token_seq[n];
        if (seq < 0) {
            pad(n);
            last_seq = -2;
            continue;
        }
        float x[VEC];
        conv_load<VEC>(c.raw + (size_t)n * c.ld + ch, x);
        if (seq != last_seq) {                   // win[j] (j >= 1) holds the input taps - j back; it moves down by one below
            const int r0 = c.cu_seqlens[seq];
            const bool fresh = c.token_pos[r0] == 0;
            const float* keep = c.keep + (size_t)c.seq_slot[seq] * (taps - 1) * c.C + ch;
#pragma unroll
            for (int j = 1; j < MAXT; ++j) {
                if (j >= taps) continue;
                const int src = n - taps + j;
#pragma unroll
                for (int v = 0; v < VEC; ++v) win[j][v] = 0.f;
                if (src >= r0) {
                    conv_load<VEC>(c.raw + (size_t)src * c.ld + ch, win[j]);
#pragma unroll
                    for (int v = 0; v < VEC; ++v) win[j][v] += b[v];
                } else if (!fresh) {
                    conv_load<VEC>(keep + (size_t)((taps - 1) + (src - r0)) * c.C, win[j]);
                }
            }
            last_seq = seq;
        }
        float y[VEC];
#pragma unroll
        for (int v = 0; v < VEC; ++v) {
            float acc = 0.f;
            x[v] += b[v];
#pragma unroll
            for (int j = 0; j < MAXT; ++j) {
                if (j + 1 < taps) win[j][v] = win[j + 1 < MAXT ? j + 1 : j][v];
                else if (j + 1 == taps) win[j][v] = x[v];
                if (j < taps) acc = fmaf(wr[j][v], win[j][v], acc);
            }
            y[v] = acc;
        }
        emit(n, y);
        if (c.keep_w != nullptr) {               // single tokens: the kept inputs (the last taps - 1 in sight) move on here
            float* keep = c.keep_w + (size_t)c.seq_slot[seq] * (taps - 1) * c.C + ch;
#pragma unroll
            for (int j = 1; j < MAXT; ++j)
                if (j < taps) conv_store<VEC>(keep + (size_t)(j - 1) * c.C, win[j]);
        }
    }
}

// How many rows a thread walks: runs as long as leave every SM several blocks; a single-token step's rows are sequences of
// their own.
inline int conv_run(int N, int blocks, bool single) {
    int run = 1;
    while (!single && run < kConvTokens && (long long)((N + 2 * run - 1) / (2 * run)) * blocks >= 4 * sm_count_cached()) run *= 2;
    return run;
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
