// Linear recurrences with a matrix state per head, S [dim keys][vdim values] in 32-bit, one kernel for three rules:
//
//   decay rule    S <- g S + beta k v^T                           o = S^T q     (g, beta per head, or per token and head)
//   delta rule    S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q  (g, beta per token and head)
//   channel rule  S <- diag(g) S + k v^T                          o = S^T q     (g per token, head and key channel)
//
// (The decay rule's beta may be left out; o may be multiplied by a constant.)  The read-out sees the current token's write.  A sequence's state lives per slot as S^T ([head][vdim][dim]: a
// thread's run of rows of one column is contiguous), starts at zero (a sequence whose first row is position 0
// ignores what the slot holds), and is carried from step to step.
//
// state_scan: one block per (sequence, head, run of value columns); a column of S is cut into R runs of DR rows,
//   one thread each (R lanes side by side, so that sums over a column are shuffles); tokens in order, a chunk of
//   them staged in shared memory while the chunk before it is walked (cp.async, two buffers).  Columns are
//   independent of one another in all rules.
//   A long sequence of the decay or the channel rule (whose state at a segment's end is linear in the state at its start,
//   cell by cell) is cut into segments that are walked side by side: first every segment from a zero state (its first
//   one from the sequence's), without read-outs, leaving its state and the product of its decays; then segment_starts
//   turns those into the states at the segments' starts, and a second walk from these makes the read-outs.
// act_rows: x logistic(x) in place on the leading columns of 32-bit rows (the decay rule's q, k, v).
// rotate_rows: rotary positions in place on the q and k heads of 32-bit rows (either pairing, the first rot_dims
//   numbers of a head; angle = position * freq in 32-bit, sincosf), the keys then multiplied by a constant.
// conv_prep (the delta rule's inputs): per token, the short causal convolution over time of the q, k, v
//   projections (per channel, `taps` wide, the last tap the current token's, the inputs before a step's first
//   row from the slot's state), x sigmoid(x) of it, q and k divided by their length per head
//   (sqrt(sum + 1e-6)), q times dim^-1/2; beta = logistic(b); g = exp(-exp(A_log) softplus(a + dt_bias)).
// conv_keep: the last taps - 1 inputs of every sequence go to the slot's state.
// conv_act_rows: the short convolution with a bias and an activation on a run of columns, many tokens to a thread; with
//   per-head step sizes: dt = softplus(raw + dt_bias) and the decay exp(-exp(A_log) dt) in the same launch.
// channel_decay: logistic(W z + b)^(1 / tau) per key channel from a low-rank row z.
#include "common.cuh"
#include "short_conv.cuh"

namespace hos {

constexpr int kScanChunk = 8;       // tokens staged at a time
constexpr int kPad = 4;             // floats after every DR staged numbers: 16-byte reads of R neighbours miss each other's banks

__device__ __forceinline__ float silu_precise(float x) { return x / (1.f + expf(-x)); }

__device__ __forceinline__ void cp_async4(void* dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit_all() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }

// x <- x logistic(x) on the first `cols` numbers of every row (the decay rule's q, k, v before the scan)
__global__ void act_rows_kernel(float* __restrict__ x, long long ld, int cols, long long n) {
    pdl_enter();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    float* p = x + (i / cols) * ld + (i % cols);
    *p = silu_precise(*p);
}

// x: float32 [N][ld]; from column 0 on `Hq` query heads and then `Hk` key heads of `dim` numbers each.  The first
// rot_dims numbers of every head turn with the token's position: style 0 pairs number i with i + rot_dims / 2,
// style 1 number 2i with 2i + 1; (u, v) -> (u cos a - v sin a, v cos a + u sin a), a = position * freq[i].  Every
// number of a key head is then multiplied by k_mult.  An item is one pair, or one number beyond rot_dims.
__global__ void __launch_bounds__(256)
rotate_rows_kernel(float* __restrict__ x, long long ld, int Hq, int Hk, int dim, int rot_dims, int style,
                   const float* __restrict__ freq, const int* __restrict__ token_pos, const int* __restrict__ token_seq,
                   float k_mult) {
    pdl_enter();
    extern __shared__ float2 rot_tab[];          // [rot_dims / 2] (sine, cosine) of this token
    const int n = blockIdx.x;
    if (token_seq[n] < 0) return;
    const float fpos = (float)token_pos[n];
    const int half = rot_dims >> 1;
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        float sn, cs;
        sincosf(fpos * freq[i], &sn, &cs);
        rot_tab[i] = make_float2(sn, cs);
    }
    __syncthreads();
    float* row = x + (size_t)n * ld;
    const int per = half + (dim - rot_dims);
    for (int it = threadIdx.x; it < (Hq + Hk) * per; it += blockDim.x) {
        const int head = it / per, j = it - head * per;
        const float m = head >= Hq ? k_mult : 1.f;
        float* hp = row + (size_t)head * dim;
        if (j < half) {
            const int a = style == 0 ? j : 2 * j, b = style == 0 ? j + half : 2 * j + 1;
            const float2 sc = rot_tab[j];
            const float u = hp[a], v = hp[b];
            hp[a] = (u * sc.y - v * sc.x) * m;
            hp[b] = (v * sc.y + u * sc.x) * m;
        } else if (m != 1.f) {
            hp[rot_dims + (j - half)] *= m;
        }
    }
}

constexpr int kDecayPerThread = 4;

// Two 32-bit multiply-adds (or products) in one instruction: each half is the plain operation with one rounding.
__device__ __forceinline__ uint64_t pair_of(float x, float y) {
    uint64_t d;
    asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(x), "f"(y));
    return d;
}
__device__ __forceinline__ void halves_of(uint64_t p, float& x, float& y) { asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(p)); }
__device__ __forceinline__ uint64_t fma_pair(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ uint64_t mul_pair(uint64_t a, uint64_t b) {
    uint64_t d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}

enum ScanRule : int { kDecayRule = 0, kDeltaRule = 1, kChannelRule = 2 };

// What a walk by segments needs: seg_len rows to a segment, `count` segments to a sequence at most (blockIdx.x is sequence x
// count + segment; count 1: the whole sequence); states: [sequences][count][H][vdim][dim]; decays: [sequences][count][H]
// (channel rule: [H][dim]).
struct Segments {
    float* states;
    float* decays;
    int len, count;
};

// A thread's cells: DR rows of DC neighbouring columns (DC > 1, the walks by segments: what is read of k, q and the decays
// serves DC columns).
template <int DR, int R, int DC, int RULE, bool LOCAL>
__global__ void __launch_bounds__(256)
state_scan_kernel(const float* __restrict__ q, const float* __restrict__ k, const float* __restrict__ v, long long ld,
                  int aligned, int act_in_walk, const float* __restrict__ g, long long g_ld, const float* __restrict__ beta,
                  long long beta_ld, float* __restrict__ state, const int* __restrict__ token_pos,
                  const int* __restrict__ token_seq, const int* __restrict__ cu_seqlens, const int* __restrict__ seq_slot,
                  float* __restrict__ out, int H, int Gk, int dim, int vdim, int CC, const float* __restrict__ rot_freq,
                  int rot_dims, int rot_style, float k_mult, float o_mult, Segments sg) {
    constexpr bool DELTA = RULE == kDeltaRule, CHANNEL = RULE == kChannelRule;
    pdl_enter();
    extern __shared__ __align__(16) float sm[];
    const int seq = blockIdx.x / sg.count, seg = blockIdx.x % sg.count, head = blockIdx.y, col0 = blockIdx.z * CC;
    int lo = cu_seqlens[seq], hi = cu_seqlens[seq + 1];
    if (hi <= lo || token_seq[lo] < 0) return;
    const bool fresh = token_pos[lo] == 0;
    bool last = true;
    if (sg.count > 1) {
        const int end = hi;
        lo += seg * sg.len;
        if (lo >= end) return;
        hi = min(end, lo + sg.len);
        last = hi == end;
        if (LOCAL && last) return;               // nothing starts from the last segment's state but the slot's, which the second walk makes
    }
    const int slot = seq_slot[seq];
    const int kh = head / (H / Gk);
    const int r = threadIdx.x % R, c = threadIdx.x / R;
    const int col = col0 + c * DC;
    const bool rot_in_walk = rot_dims > 0 || k_mult != 1.f;
    const int n_cols = CC / DC;                  // threads' columns of this block
    auto live = [&](int j) { return c < n_cols && col + j < vdim; };
    const int dpad = R * (DR + kPad);
    // two buffers of staged tokens: while one chunk is walked the next one's rows are on their way (cp.async)
    const int per_buf = kScanChunk * ((CHANNEL ? 3 : 2) * dpad + 2 * CC) + 2 * kScanChunk;      // q, k, (g,) v, o, g, beta
    const bool v_aligned = DC == 4 && (vdim & 3) == 0 && (ld & 3) == 0 && ((uintptr_t)v & 15) == 0;
    const bool v_scaled = RULE == kDecayRule && beta != nullptr;

    float S[DC][DR];
    const size_t cell = ((size_t)head * vdim + (live(0) ? col : 0)) * dim + r * DR, cells = (size_t)H * vdim * dim;
    float* st = state + (size_t)slot * cells + cell;                                  // the slot's
    float* seg_st = sg.states + ((size_t)seq * sg.count + seg) * cells + cell;        // the segment's, where there are several
    // where this walk starts: the slot's state (whole sequences, and the first segment of a first walk), zero, or the
    // segment's start
    const bool from_seg = sg.count > 1 && !LOCAL;
    const float* src = from_seg ? seg_st : st;
    const bool zero = from_seg ? false : (fresh || seg > 0);
    // a thread's run of rows is contiguous in the kept S^T: 16 bytes at a time where the run is whole and aligned
    const bool whole = r * DR + DR <= dim && (dim & 3) == 0;
#pragma unroll
    for (int j = 0; j < DC; ++j) {
        const float* from = src + (size_t)j * dim;
        if (!zero && whole && live(j)) {
#pragma unroll
            for (int i = 0; i < DR / 4; ++i) {
                const float4 t = ((const float4*)from)[i];
                S[j][4 * i] = t.x; S[j][4 * i + 1] = t.y; S[j][4 * i + 2] = t.z; S[j][4 * i + 3] = t.w;
            }
        } else {
#pragma unroll
            for (int i = 0; i < DR; ++i) S[j][i] = (!zero && live(j) && r * DR + i < dim) ? from[i] : 0.f;
        }
    }
    uint64_t P[DC][DR / 2];                      // four columns: the cells as pairs of rows
    if (DC == 4) {
#pragma unroll
        for (int j = 0; j < DC; ++j)
#pragma unroll
            for (int i = 0; i < DR / 2; ++i) P[j][i] = pair_of(S[j][2 * i], S[j][2 * i + 1]);
    }
    // rows beyond dim and columns beyond vdim are read by the walk and never staged: they stay zero for good
    if (R * DR != dim || col0 + CC > vdim) {
        for (int i = threadIdx.x; i < 2 * per_buf; i += blockDim.x) sm[i] = 0.f;
        __syncthreads();
    }

    auto stage = [&](int t0, int nt, float* buf) {
        float* qs = buf;
        float* ks = qs + kScanChunk * dpad;
        float* gk = ks + kScanChunk * dpad;          // the channel rule's decays, laid out as the keys
        float* vs = ks + (CHANNEL ? 2 : 1) * kScanChunk * dpad;
        float* gs = vs + 2 * kScanChunk * CC;        // after v and o
        float* bs = gs + kScanChunk;
        if (aligned) {
            const int d4 = dim >> 2;
            for (int idx = threadIdx.x; idx < nt * d4; idx += blockDim.x) {
                const int t = idx / d4, d = (idx % d4) << 2;
                const int at = t * dpad + d + (d / DR) * kPad;
                if (!LOCAL) cp_async16(qs + at, q + (size_t)(t0 + t) * ld + kh * dim + d);
                cp_async16(ks + at, k + (size_t)(t0 + t) * ld + kh * dim + d);
                if (CHANNEL) cp_async16(gk + at, g + (size_t)(t0 + t) * g_ld + head * dim + d);
            }
        } else {
            for (int idx = threadIdx.x; idx < nt * dim; idx += blockDim.x) {
                const int t = idx / dim, d = idx % dim;
                const int at = t * dpad + d + (d / DR) * kPad;
                if (!LOCAL) cp_async4(qs + at, q + (size_t)(t0 + t) * ld + kh * dim + d);
                cp_async4(ks + at, k + (size_t)(t0 + t) * ld + kh * dim + d);
                if (CHANNEL) cp_async4(gk + at, g + (size_t)(t0 + t) * g_ld + head * dim + d);
            }
        }
        const int ncol = min(CC, vdim - col0);
        if (DC == 4 && v_aligned) {
            const int c4 = ncol >> 2;
            for (int idx = threadIdx.x; idx < nt * c4; idx += blockDim.x) {
                const int t = idx / c4, cc = (idx % c4) << 2;
                cp_async16(vs + t * CC + cc, v + (size_t)(t0 + t) * ld + head * vdim + col0 + cc);
            }
        } else
        for (int idx = threadIdx.x; idx < nt * ncol; idx += blockDim.x) {
            const int t = idx / ncol, cc = idx % ncol;
            cp_async4(vs + t * CC + cc, v + (size_t)(t0 + t) * ld + head * vdim + col0 + cc);
        }
        if (threadIdx.x < nt) {
            if (!CHANNEL) cp_async4(gs + threadIdx.x, g + (size_t)(t0 + threadIdx.x) * g_ld + head);
            if (DELTA || v_scaled) cp_async4(bs + threadIdx.x, beta + (size_t)(t0 + threadIdx.x) * beta_ld + head);
        }
        cp_async_commit_all();
    };

    stage(lo, min(kScanChunk, hi - lo), sm);
    int which = 0;
    float dec[kDecayPerThread] = {1.f, 1.f, 1.f, 1.f};       // first walks: the product of the segment's decays
    for (int t0 = lo; t0 < hi; t0 += kScanChunk, which ^= 1) {
        const int nt = min(kScanChunk, hi - t0);
        cp_async_wait_all();
        __syncthreads();            // this chunk has landed; everyone is done with the other buffer
        if (t0 + kScanChunk < hi) stage(t0 + kScanChunk, min(kScanChunk, hi - t0 - kScanChunk), sm + (which ^ 1) * per_buf);
        float* qs = sm + which * per_buf;
        float* ks = qs + kScanChunk * dpad;
        if (!LOCAL && rot_in_walk) {
            // the staged q and k turn with their tokens' positions, and the keys take their factor, as rotate_rows would
            // have done in a launch of its own (meant for single-token steps: every block of a head repeats it)
            const int half = rot_dims >> 1, per = half + (dim - rot_dims);
            for (int idx = threadIdx.x; idx < nt * per; idx += blockDim.x) {
                const int t = idx / per, j = idx - t * per;
                float* qp = qs + t * dpad;
                float* kp = ks + t * dpad;
                if (j < half) {
                    const int a = rot_style == 0 ? j : 2 * j, b = rot_style == 0 ? j + half : 2 * j + 1;
                    const int ia = a + (a / DR) * kPad, ib = b + (b / DR) * kPad;
                    float sn, cs;
                    sincosf((float)token_pos[t0 + t] * rot_freq[j], &sn, &cs);
                    const float qu = qp[ia], qv = qp[ib], ku = kp[ia], kv = kp[ib];
                    qp[ia] = qu * cs - qv * sn;
                    qp[ib] = qv * cs + qu * sn;
                    kp[ia] = (ku * cs - kv * sn) * k_mult;
                    kp[ib] = (kv * cs + ku * sn) * k_mult;
                } else {
                    const int d = rot_dims + (j - half);
                    kp[d + (d / DR) * kPad] *= k_mult;
                }
            }
            __syncthreads();
        }
        float* gk = ks + kScanChunk * dpad;
        float* vs = ks + (CHANNEL ? 2 : 1) * kScanChunk * dpad;
        float* os = vs + kScanChunk * CC;
        float* gs = os + kScanChunk * CC;
        float* bs = gs + kScanChunk;
        if constexpr (DC == 4) {
#pragma unroll 2
            for (int t = 0; t < nt; ++t) {
                const float4* k4 = (const float4*)(ks + t * dpad + r * (DR + kPad));
                const float4* q4 = (const float4*)(qs + t * dpad + r * (DR + kPad));
                const float4* g4 = (const float4*)(gk + t * dpad + r * (DR + kPad));
                float4 u = c < n_cols ? *(const float4*)(vs + t * CC + c * DC) : make_float4(0.f, 0.f, 0.f, 0.f);
                if (v_scaled) {
                    const float f = bs[t];
                    u = make_float4(u.x * f, u.y * f, u.z * f, u.w * f);
                }
                const uint64_t uu[4] = {pair_of(u.x, u.x), pair_of(u.y, u.y), pair_of(u.z, u.z), pair_of(u.w, u.w)};
                const uint64_t gt = CHANNEL ? 0 : pair_of(gs[t], gs[t]);
                uint64_t a[4] = {0, 0, 0, 0};
#pragma unroll
                for (int i = 0; i < DR / 4; ++i) {
                    const float4 kk = k4[i];
                    const uint64_t k2[2] = {pair_of(kk.x, kk.y), pair_of(kk.z, kk.w)};
                    uint64_t g2[2] = {gt, gt}, q2[2] = {0, 0};
                    if (CHANNEL) {
                        const float4 gg = g4[i];
                        g2[0] = pair_of(gg.x, gg.y);
                        g2[1] = pair_of(gg.z, gg.w);
                    }
                    if (!LOCAL) {
                        const float4 qq = q4[i];
                        q2[0] = pair_of(qq.x, qq.y);
                        q2[1] = pair_of(qq.z, qq.w);
                    }
#pragma unroll
                    for (int e = 0; e < 2; ++e)
#pragma unroll
                        for (int j = 0; j < 4; ++j) {
                            uint64_t& p = P[j][2 * i + e];
                            p = fma_pair(g2[e], p, mul_pair(k2[e], uu[j]));
                            if (!LOCAL) a[j] = fma_pair(p, q2[e], a[j]);
                        }
                }
                if (LOCAL) continue;
                // four columns' sums over R threads: a thread hands on the columns it does not end with, two and then one,
                // and the rest of the threads add up the one that is left
                static_assert(R >= 4, "the sums of four columns");
                float p[4];
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    float x, y;
                    halves_of(a[j], x, y);
                    p[j] = x + y;
                }
                const bool up = (r & (R / 2)) != 0, up2 = (r & (R / 4)) != 0;
                const float x0 = __shfl_xor_sync(0xffffffffu, up ? p[0] : p[2], R / 2);
                const float x1 = __shfl_xor_sync(0xffffffffu, up ? p[1] : p[3], R / 2);
                const float y0 = (up ? p[2] : p[0]) + x0, y1 = (up ? p[3] : p[1]) + x1;
                float acc = (up2 ? y1 : y0) + __shfl_xor_sync(0xffffffffu, up2 ? y0 : y1, R / 4);
#pragma unroll
                for (int o = R / 8; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
                if ((r & (R / 4 - 1)) == 0 && c < n_cols) os[t * CC + c * DC + (up ? 2 : 0) + (up2 ? 1 : 0)] = acc * o_mult;
            }
        } else {       // every thread walks (a warp's shuffles want all its lanes); only live columns are written
            float part[kScanChunk];       // the read-outs' partial sums: added up after the walk, off its chain
#pragma unroll
            for (int t = 0; t < kScanChunk; ++t) {
                part[t] = 0.f;
                if (t >= nt) continue;
                const float4* k4 = (const float4*)(ks + t * dpad + r * (DR + kPad));
                const float4* q4 = (const float4*)(qs + t * dpad + r * (DR + kPad));
                const float4* g4 = (const float4*)(gk + t * dpad + r * (DR + kPad));
                const float gt = CHANNEL ? 0.f : gs[t];
                float u = c < n_cols ? vs[t * CC + c] : 0.f;
                if (RULE == kDecayRule && act_in_walk) u = silu_precise(u);      // single tokens: the activation rides here
                if (v_scaled) u *= bs[t];
                if (DELTA) {
                    float d0 = 0.f, d1 = 0.f, d2 = 0.f, d3 = 0.f;       // four chains, not one of DR links
#pragma unroll
                    for (int i = 0; i < DR / 4; ++i) {
                        const float4 kk = k4[i];
                        S[0][4 * i] *= gt; S[0][4 * i + 1] *= gt; S[0][4 * i + 2] *= gt; S[0][4 * i + 3] *= gt;
                        d0 = fmaf(S[0][4 * i], kk.x, d0);
                        d1 = fmaf(S[0][4 * i + 1], kk.y, d1);
                        d2 = fmaf(S[0][4 * i + 2], kk.z, d2);
                        d3 = fmaf(S[0][4 * i + 3], kk.w, d3);
                    }
                    float dot = (d0 + d1) + (d2 + d3);
#pragma unroll
                    for (int o = 1; o < R; o <<= 1) dot += __shfl_xor_sync(0xffffffffu, dot, o);
                    u = bs[t] * (u - dot);
                }
                float a[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                for (int i = 0; i < DR / 4; ++i) {
                    float4 kk = k4[i], qq = LOCAL ? make_float4(0.f, 0.f, 0.f, 0.f) : q4[i];
                    if (RULE == kDecayRule && act_in_walk) {
                        kk = make_float4(silu_precise(kk.x), silu_precise(kk.y), silu_precise(kk.z), silu_precise(kk.w));
                        qq = make_float4(silu_precise(qq.x), silu_precise(qq.y), silu_precise(qq.z), silu_precise(qq.w));
                    }
                    const float4 gg = CHANNEL ? g4[i] : make_float4(gt, gt, gt, gt);
                    float* s4 = &S[0][4 * i];
                    if (DELTA) {
                        s4[0] = fmaf(kk.x, u, s4[0]);
                        s4[1] = fmaf(kk.y, u, s4[1]);
                        s4[2] = fmaf(kk.z, u, s4[2]);
                        s4[3] = fmaf(kk.w, u, s4[3]);
                    } else {
                        s4[0] = fmaf(gg.x, s4[0], kk.x * u);
                        s4[1] = fmaf(gg.y, s4[1], kk.y * u);
                        s4[2] = fmaf(gg.z, s4[2], kk.z * u);
                        s4[3] = fmaf(gg.w, s4[3], kk.w * u);
                    }
                    if (LOCAL) continue;
                    a[0] = fmaf(s4[0], qq.x, a[0]);
                    a[1] = fmaf(s4[1], qq.y, a[1]);
                    a[2] = fmaf(s4[2], qq.z, a[2]);
                    a[3] = fmaf(s4[3], qq.w, a[3]);
                }
                part[t] = (a[0] + a[1]) + (a[2] + a[3]);
            }
#pragma unroll
            for (int t = 0; t < kScanChunk; ++t) {
                if (LOCAL || t >= nt) break;
                float acc = part[t];
#pragma unroll
                for (int o = 1; o < R; o <<= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
                if (r == 0 && c < CC) os[t * CC + c] = acc * o_mult;
            }
        }
        if (LOCAL) {
            if (blockIdx.z == 0) {
#pragma unroll
                for (int i = 0; i < kDecayPerThread; ++i) {
                    const int d = threadIdx.x + i * blockDim.x;
                    if (d >= (CHANNEL ? dim : 1)) break;
                    for (int t = 0; t < nt; ++t) dec[i] *= CHANNEL ? gk[t * dpad + d + (d / DR) * kPad] : gs[t];
                }
            }
            continue;
        }
        __syncthreads();
        for (int idx = threadIdx.x; idx < nt * CC; idx += blockDim.x) {
            const int t = idx / CC, cc = idx % CC;
            if (col0 + cc < vdim) out[((size_t)(t0 + t) * H + head) * vdim + col0 + cc] = os[idx];
        }
    }
    if (LOCAL) {
        if (blockIdx.z == 0) {
            float* dp = sg.decays + (((size_t)seq * sg.count + seg) * H + head) * (CHANNEL ? dim : 1);
#pragma unroll
            for (int i = 0; i < kDecayPerThread; ++i) {
                const int d = threadIdx.x + i * blockDim.x;
                if (d < (CHANNEL ? dim : 1)) dp[d] = dec[i];
            }
        }
        st = seg_st;
    } else if (!last) {
        return;                                  // only the last segment's state is the sequence's
    }
    if (DC == 4) {
#pragma unroll
        for (int j = 0; j < DC; ++j)
#pragma unroll
            for (int i = 0; i < DR / 2; ++i) halves_of(P[j][i], S[j][2 * i], S[j][2 * i + 1]);
    }
#pragma unroll
    for (int j = 0; j < DC; ++j) {
        if (!live(j)) continue;
        float* to = st + (size_t)j * dim;
        if (whole) {
#pragma unroll
            for (int i = 0; i < DR / 4; ++i)
                ((float4*)to)[i] = make_float4(S[j][4 * i], S[j][4 * i + 1], S[j][4 * i + 2], S[j][4 * i + 3]);
        } else {
#pragma unroll
            for (int i = 0; i < DR; ++i)
                if (r * DR + i < dim) to[i] = S[j][i];
        }
    }
}

// states: what the first walk left, [count][cells] per sequence; becomes the states at the segments' starts (the first one's:
// the slot's, or zero).  A thread per cell; decays: a number per head, or (channel) per head and key number.
__global__ void __launch_bounds__(256)
segment_starts_kernel(const float* __restrict__ state, Segments sg, const int* __restrict__ token_pos, const int* __restrict__ token_seq,
                      const int* __restrict__ cu_seqlens, const int* __restrict__ seq_slot, int H, int dim, int vdim, int channel) {
    pdl_enter();
    const int seq = blockIdx.y;
    const int lo = cu_seqlens[seq], len = cu_seqlens[seq + 1] - lo;
    if (len <= 0 || token_seq[lo] < 0) return;
    const long long cells = (long long)H * vdim * dim;
    const long long cell = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (cell >= cells) return;
    const int n = (len + sg.len - 1) / sg.len;
    const int head = (int)(cell / ((long long)vdim * dim));
    const int per = channel ? H * dim : H, at = channel ? head * dim + (int)(cell % dim) : head;
    float* st = sg.states + (size_t)seq * sg.count * cells + cell;
    const float* dp = sg.decays + (size_t)seq * sg.count * per + at;
    float cur = token_pos[lo] == 0 ? 0.f : state[(size_t)seq_slot[seq] * cells + cell];
    constexpr int B = 8;                          // loads under way together
    for (int s0 = 0; s0 < n; s0 += B) {
        float local[B], d[B];
#pragma unroll
        for (int i = 0; i < B; ++i) {
            const int s = s0 + i;
            const bool in = s < n - 1;            // the last segment has left nothing
            local[i] = in ? st[(size_t)s * cells] : 0.f;
            d[i] = in ? dp[(size_t)s * per] : 0.f;
        }
#pragma unroll
        for (int i = 0; i < B; ++i) {
            const int s = s0 + i;
            if (s >= n) break;
            st[(size_t)s * cells] = cur;
            cur = s == 0 ? local[i] : fmaf(d[i], cur, local[i]);      // the first segment's walk began with the sequence's state
        }
    }
}

// raw: float32 [N][ld]: q (Gk * dim) | k (Gk * dim) | v (H * vdim) | b (H) | a (H) | ... ; conv_w: [C][taps] over
// the first C = 2 Gk dim + H vdim columns; conv_state: [slots][taps - 1][C], row j the input taps - 1 - j tokens back.
__global__ void __launch_bounds__(256)
conv_prep_kernel(const float* __restrict__ raw, long long ld, const float* __restrict__ conv_w, int taps,
                 const float* conv_state,      // may be written through keep_here: neither is __restrict__
                 const float* __restrict__ a_log, const float* __restrict__ dt_bias,
                 const int* __restrict__ token_pos, const int* __restrict__ token_seq, const int* __restrict__ cu_seqlens,
                 const int* __restrict__ seq_slot, float* __restrict__ act, float* __restrict__ beta_out,
                 float* __restrict__ g_out, int H, int Gk, int dim, int vdim, float* keep_here) {
    pdl_enter();
    extern __shared__ float qk[];                // [2 Gk dim] after the activation
    __shared__ float inv_len[64];
    const int n = blockIdx.x;
    const int seq = token_seq[n];
    const int QK = 2 * Gk * dim, C = QK + H * vdim;
    float* arow = act + (size_t)n * C;
    if (seq < 0) {
        for (int i = threadIdx.x; i < C; i += blockDim.x) arow[i] = 0.f;
        for (int i = threadIdx.x; i < H; i += blockDim.x) {
            beta_out[(size_t)n * H + i] = 0.f;
            g_out[(size_t)n * H + i] = 1.f;
        }
        return;
    }
    const int r0 = cu_seqlens[seq];
    const bool fresh = token_pos[r0] == 0;
    const float* keep = conv_state + (size_t)seq_slot[seq] * (taps - 1) * C;
    // keep_here: every sequence of the step brings one token, so this block alone reads and writes its slot's kept
    // inputs (a thread the channels it convolves): they move on by one here instead of in a launch of their own
    float* keep_w = keep_here != nullptr ? keep_here + (size_t)seq_slot[seq] * (taps - 1) * C : nullptr;
    for (int ch = threadIdx.x; ch < C; ch += blockDim.x) {
        const float acc = short_conv(raw + ch, ld, 0.f, conv_w, taps, keep, keep_w, C, ch, n, r0, fresh);
        const float y = silu_precise(acc);
        if (ch < QK) qk[ch] = y;
        else arow[ch] = y;
    }
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarps = blockDim.x >> 5;
    for (int hd0 = 0; hd0 < 2 * Gk; hd0 += 64) {         // the heads' lengths, a warp per head
        for (int hd = hd0 + warp; hd < min(2 * Gk, hd0 + 64); hd += nwarps) {
            float ss = 0.f;
            for (int d = lane; d < dim; d += 32) ss = fmaf(qk[hd * dim + d], qk[hd * dim + d], ss);
            ss = warp_sum(ss);
            if (lane == 0) inv_len[hd - hd0] = (1.f / sqrtf(ss + 1e-6f)) * (hd < Gk ? 1.f / sqrtf((float)dim) : 1.f);
        }
        __syncthreads();
        for (int i = hd0 * dim + threadIdx.x; i < min(2 * Gk, hd0 + 64) * dim; i += blockDim.x)
            arow[i] = qk[i] * inv_len[i / dim - hd0];
        __syncthreads();
    }
    for (int h = threadIdx.x; h < H; h += blockDim.x) {
        const float b = raw[(size_t)n * ld + C + h], a = raw[(size_t)n * ld + C + H + h] + dt_bias[h];
        beta_out[(size_t)n * H + h] = 1.f / (1.f + expf(-b));
        const float sp = a > 20.f ? a : log1pf(expf(a));
        g_out[(size_t)n * H + h] = expf(-expf(a_log[h]) * sp);
    }
}

// act(x): 0 none, 1 x logistic(x)
__device__ __forceinline__ float conv_act(float x, int act) { return act == 1 ? silu_precise(x) : x; }

// out[n][c] = act(convolution + bias[c]) for C columns of 32-bit rows (conv_walk in short_conv.cuh).  The last block of a row
// run takes the per-head step sizes: dt = softplus(raw + dt_bias), decay = exp(-exp(A_log) dt).
template <int TAPS, int VEC>
__global__ void __launch_bounds__(128)
conv_act_rows_kernel(ConvWalk c, const float* __restrict__ bias, int act, float* __restrict__ out, int N, int run, int conv_blocks,
                     const float* __restrict__ dt_raw, const float* __restrict__ dt_bias, const float* __restrict__ a_log,
                     float* __restrict__ dt_out, float* __restrict__ g_out, int H) {
    pdl_enter();
    const int n0 = blockIdx.y * run, n1 = min(N, n0 + run);
    if ((int)blockIdx.x >= conv_blocks) {
        for (int i = threadIdx.x; i < (n1 - n0) * H; i += blockDim.x) {
            const int n = n0 + i / H, h = i % H;
            float dt = 0.f, g = 1.f;
            if (c.token_seq[n] >= 0) {
                const float a = dt_raw[(size_t)n * c.ld + h] + dt_bias[h];
                dt = a > 20.f ? a : log1pf(expf(a));
                g = expf(-expf(a_log[h]) * dt);
            }
            dt_out[(size_t)n * H + h] = dt;
            g_out[(size_t)n * H + h] = g;
        }
        return;
    }
    const int ch = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
    if (ch >= c.C) return;
    float b[VEC];
#pragma unroll
    for (int v = 0; v < VEC; ++v) b[v] = bias != nullptr ? bias[ch + v] : 0.f;
    conv_walk<TAPS, VEC>(
        c, ch, n0, n1,
        [&](int n, float (&y)[VEC]) {
#pragma unroll
            for (int v = 0; v < VEC; ++v) y[v] = conv_act(y[v] + b[v], act);
            conv_store<VEC>(out + (size_t)n * c.C + ch, y);
        },
        [&](int n) {
            float y[VEC];
#pragma unroll
            for (int v = 0; v < VEC; ++v) y[v] = 0.f;
            conv_store<VEC>(out + (size_t)n * c.C + ch, y);
        });
}

// out[n][c] = logistic(z)^(1 / tau), z = sum_r w[c][r] low[n][r] + b[c]: exp(-softplus(-z) / tau), 32-bit.  A block takes
// kDecayRows rows and 128 channels; the low-rank rows are staged in shared memory.
constexpr int kDecayRows = 8;
__global__ void __launch_bounds__(128)
channel_decay_kernel(const float* __restrict__ low, long long ld, const float* __restrict__ w, const float* __restrict__ b,
                     int rank, float inv_tau, float* __restrict__ out, int N, int C) {
    pdl_enter();
    extern __shared__ float low_s[];             // [kDecayRows][rank]
    const int n0 = blockIdx.y * kDecayRows, rows = min(kDecayRows, N - n0);
    for (int i = threadIdx.x; i < kDecayRows * rank; i += blockDim.x) {
        const int r = i / rank;
        low_s[i] = r < rows ? low[(size_t)(n0 + r) * ld + i % rank] : 0.f;
    }
    __syncthreads();
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= C) return;
    float acc[kDecayRows];
#pragma unroll
    for (int r = 0; r < kDecayRows; ++r) acc[r] = b[c];
    for (int k = 0; k < rank; ++k) {
        const float wv = w[(size_t)k * C + c];   // [rank][C]: neighbouring channels side by side
#pragma unroll
        for (int r = 0; r < kDecayRows; ++r) acc[r] = fmaf(wv, low_s[r * rank + k], acc[r]);
    }
#pragma unroll
    for (int r = 0; r < kDecayRows; ++r) {
        if (r >= rows) break;
        const float z = acc[r];
        const float sp = fmaxf(-z, 0.f) + log1pf(expf(-fabsf(z)));      // softplus(-z) without overflow
        out[(size_t)(n0 + r) * C + c] = expf(-sp * inv_tau);
    }
}

}  // namespace hos

using namespace hos;

namespace hos {
// How a walk is cut: DR rows of a column to a thread, R threads to a column, CC columns to a block.
struct ScanShape {
    int DR, R, CC, DC = 1;
    ScanShape(int dim, int vdim, bool segments = false) {
        // short runs of rows per thread: a token's walk is a chain of dependent instructions (scale, dot, sum over the
        // runs, update, read-out, sum), and with few (sequence, head) pairs nothing else hides its latency; the sums over
        // 16 or 32 runs are shuffles
        // (heads of 128 x 128, 2,048 tokens, decay / delta rule: 4 rows to a thread 477 / 628 us, 8 rows 459 / 598, 16 rows
        // 584 / 679, 32 rows 900 / 961)
        DR = dim <= 16 ? 4 : (dim <= 256 ? 8 : (dim <= 512 ? 16 : 32));
        R = 1;
        while (R * DR < dim) R <<= 1;
        if (DR == 8 && R < 4) R = 4;          // the compiled shapes (rows beyond dim are zeros)
        if (DR >= 16) R = 32;
        if (segments && DR == 8) DC = 4;      // the shapes that are compiled for four columns to a thread
        CC = 256 / R * DC;
        if (CC > vdim) CC = (vdim + DC - 1) / DC * DC;
    }
    int threads() const { return (CC / DC * R + 31) / 32 * 32; }
};
constexpr int kMinSegment = 64;       // tokens
}  // namespace hos

// How many tokens a segment has where sequences that bring up to max_new tokens are worth walking in segments (see the file's
// head); 0 where they are not.  The caller then gives hos_state_scan the workspace: with n = ceil(max_new / that),
// n_seqs * n * H * vdim * dim and n_seqs * n * H (channel rule: H * dim) floats.
extern "C" int hos_state_scan_segment(int n_seqs, int H, int dim, int vdim, int max_new, int rule) {
    if (rule == kDeltaRule || n_seqs <= 0 || max_new < 3 * kMinSegment || dim <= 0 || dim > 1024 || vdim <= 0) return 0;
    const ScanShape shape(dim, vdim, true);
    if (rule == kChannelRule && dim > kDecayPerThread * shape.threads()) return 0;
    const long long blocks = (long long)n_seqs * H * ((vdim + shape.CC - 1) / shape.CC);
    // a walk is bound by its chain until several blocks share an SM; two walks instead of one must be paid for
    // (four columns to a thread, 2,048 tokens, 64 / 128 heads of 128 x 64: 4 blocks wanted to an SM 388 / 759 us, 3 421 / 824)
    const long long want = (shape.DC > 1 ? 4ll : 8ll) * sm_count_cached() / blocks;
    if (want < 3) return 0;
    const int count = (int)(want < max_new / kMinSegment ? want : max_new / kMinSegment);
    const int len = (max_new + count - 1) / count;
    return (len + kScanChunk - 1) / kScanChunk * kScanChunk;
}

// q, k: rows of Gk heads of `dim` numbers; v: rows of H heads of `vdim`; all float32 with `ld` numbers between rows.
// rule: 0 decay, 1 delta, 2 channel.  g: [.][H] (channel rule: [.][H * dim]) with g_ld between rows (0: one row of constants).
// beta: the delta rule's; with the decay rule, if given, the factor on v; o_mult: a constant on the read-outs.  state: [slots][H][vdim][dim].
// out: float32 [N][H][vdim].  act_in_walk (decay rule only, meant for single-token steps): q, k, v are taken through
// x logistic(x) as they are read, instead of by hos_act_rows before.  rot_freq ([rot_dims / 2], or null), rot_style, k_mult:
// the staged q and k are turned by their tokens' positions and the keys multiplied, as hos_rotate_rows would have done
// before (meant for single-token steps; it follows the rows as they are, so it does not go with act_in_walk).  seg_len, seg_count > 1: the
// walk in segments (hos_state_scan_segment), seg_count of them to a sequence at most, with its workspace.
extern "C" int hos_state_scan(const float* q, const float* k, const float* v, long long ld, int act_in_walk, int rule,
                              float o_mult, const float* g, long long g_ld, const float* beta, long long beta_ld, float* state, const int* token_pos,
                              const int* token_seq, const int* cu_seqlens, const int* seq_slot, float* out, int n_rows,
                              int n_seqs, int H, int Gk, int dim, int vdim, const float* rot_freq, int rot_dims, int rot_style,
                              float k_mult, int seg_len, int seg_count, float* seg_states, float* seg_decays, cudaStream_t stream) {
    if (n_seqs <= 0) return 0;
    if (rot_freq == nullptr) rot_dims = 0;
    if (rot_dims < 0 || rot_dims % 2 != 0 || rot_dims > dim || (rot_style != 0 && rot_style != 1))
        HOS_REFUSE("state_scan: %d rotated numbers in heads of %d", rot_dims, dim);
    if (Gk <= 0 || H % Gk != 0) HOS_REFUSE("state_scan: %d heads are not a multiple of %d key heads", H, Gk);
    if (dim <= 0 || dim > 1024 || vdim <= 0) HOS_REFUSE("state_scan: heads of %d x %d", dim, vdim);
    const bool segments = seg_count > 1;
    const ScanShape shape(dim, vdim, segments);
    const int DR = shape.DR, R = shape.R, DC = shape.DC;
    int CC = shape.CC;
    // single tokens and few (sequence, head) pairs: fewer columns to a block, so that the blocks fill the GPU (columns
    // are independent; every block stages the whole q and k rows, which a long walk would pay for token by token)
    if (n_rows <= 2 * n_seqs && !segments)
        while (CC * R > 64 && (long long)n_seqs * H * ((vdim + CC - 1) / CC) < 2 * sm_count_cached()) CC = (CC + 1) / 2;
    const int threads = (CC / DC * R + 31) / 32 * 32;
    const int dpad = R * (DR + kPad);
    if (segments && (rule == kDeltaRule || act_in_walk || rot_dims > 0 || k_mult != 1.f || seg_len <= 0 || seg_states == nullptr ||
                     seg_decays == nullptr || (rule == kChannelRule && dim > kDecayPerThread * threads)))
        HOS_REFUSE("state_scan: %d segments of %d tokens do not fit this walk", seg_count, seg_len);
    const Segments sg{seg_states, seg_decays, segments ? seg_len : 1, segments ? seg_count : 1};
    if (rule < kDecayRule || rule > kChannelRule || (rule == kDeltaRule && beta == nullptr) || (rule == kChannelRule && beta != nullptr))
        HOS_REFUSE("state_scan: rule %d and its inputs do not fit", rule);
    if (rule == kChannelRule && Gk != H) HOS_REFUSE("state_scan: the channel rule has a key head per head");
    const int wide_rows = rule == kChannelRule ? 3 : 2;
    const size_t smem = (size_t)2 * (wide_rows * kScanChunk * dpad + 2 * kScanChunk * CC + 2 * kScanChunk) * sizeof(float);
    const int aligned = (dim % 4 == 0 && ld % 4 == 0 && (uintptr_t)q % 16 == 0 && (uintptr_t)k % 16 == 0 &&
                         (rule != kChannelRule || (g_ld % 4 == 0 && (uintptr_t)g % 16 == 0))) ? 1 : 0;
    const dim3 grid(n_seqs * sg.count, H, (vdim + CC - 1) / CC);
    if (rule != kDecayRule && act_in_walk) HOS_REFUSE("state_scan: the activation in the walk is the decay rule's");
    if (smem > 200 * 1024) HOS_REFUSE("state_scan: heads of %d x %d do not fit a block's shared memory", dim, vdim);
#define HOS_SCAN(DRv, Rv, DCv, DL, LOC)                                                                                   \
    do {                                                                                                             \
        if (smem > 48 * 1024)                                                                                        \
            cudaFuncSetAttribute(state_scan_kernel<DRv, Rv, DCv, DL, LOC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        launch_pdl(state_scan_kernel<DRv, Rv, DCv, DL, LOC>, grid, dim3(threads), smem, stream, q, k, v, ld, aligned, act_in_walk, g, g_ld, beta, \
                   beta_ld, state, token_pos, token_seq, cu_seqlens, seq_slot, out, H, Gk, dim, vdim, CC, rot_freq,  \
                   rot_dims, rot_style, k_mult, o_mult, sg);                                                         \
    } while (0)
#define HOS_SCAN_S(DRv, Rv, DL)                                                                                      \
    do {                                                                                                             \
        constexpr int DCs = DRv == 8 ? 4 : 1;                                                                        \
        if (segments) {                                                                                              \
            HOS_SCAN(DRv, Rv, DCs, DL, true);                                                                           \
            launch_pdl(segment_starts_kernel, dim3((unsigned)(((long long)H * vdim * dim + 255) / 256), n_seqs), dim3(256), 0, stream, \
                       (const float*)state, sg, token_pos, token_seq, cu_seqlens, seq_slot, H, dim, vdim, DL == kChannelRule ? 1 : 0); \
            HOS_SCAN(DRv, Rv, DCs, DL, false);                                                                       \
        } else {                                                                                                     \
            HOS_SCAN(DRv, Rv, 1, DL, false);                                                                         \
        }                                                                                                            \
    } while (0)
#define HOS_SCAN_D(DRv, Rv)                                                                                          \
    do {                                                                                                             \
        if (rule == kDeltaRule) HOS_SCAN(DRv, Rv, 1, kDeltaRule, false);                                              \
        else if (rule == kChannelRule) HOS_SCAN_S(DRv, Rv, kChannelRule);                                            \
        else HOS_SCAN_S(DRv, Rv, kDecayRule);                                                                        \
    } while (0)
    // the shapes that the choice of DR above can give: (4; 1, 2, 4), (8; 4 to 32), (16; 32), (32; 32)
    if (DR == 4 && R == 1) HOS_SCAN_D(4, 1);
    else if (DR == 4 && R == 2) HOS_SCAN_D(4, 2);
    else if (DR == 4) HOS_SCAN_D(4, 4);
    else if (DR == 8 && R <= 4) HOS_SCAN_D(8, 4);
    else if (DR == 8 && R == 8) HOS_SCAN_D(8, 8);
    else if (DR == 8 && R == 16) HOS_SCAN_D(8, 16);
    else if (DR == 8) HOS_SCAN_D(8, 32);
    else if (DR == 16) HOS_SCAN_D(16, 32);
    else HOS_SCAN_D(32, 32);
#undef HOS_SCAN_D
#undef HOS_SCAN_S
#undef HOS_SCAN
    return check_launch("state_scan");
}

extern "C" int hos_act_rows(float* x, long long ld, int cols, int N, cudaStream_t stream) {
    const long long n = (long long)N * cols;
    if (n <= 0) return 0;
    launch_pdl(act_rows_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, stream, x, ld, cols, n);
    return check_launch("act_rows");
}

// x: float32 rows of ld numbers whose first (Hq + Hk) * dim columns are the query heads and then the key heads; freq:
// [rot_dims / 2] or null (no rotation: only the keys' multiplier is applied); style 0: halves, 1: neighbours.
extern "C" int hos_rotate_rows(float* x, long long ld, int Hq, int Hk, int dim, int rot_dims, int style, const float* freq,
                               const int* token_pos, const int* token_seq, float k_mult, int N, cudaStream_t stream) {
    if (N <= 0 || Hq + Hk <= 0) return 0;
    if (freq == nullptr) rot_dims = 0;
    if (rot_dims < 0 || rot_dims % 2 != 0 || rot_dims > dim) HOS_REFUSE("rotate_rows: %d rotated numbers in heads of %d", rot_dims, dim);
    if (style != 0 && style != 1) HOS_REFUSE("rotate_rows: unknown pairing %d", style);
    if (rot_dims == 0 && k_mult == 1.f) return 0;
    const size_t smem = (size_t)(rot_dims / 2 + 1) * sizeof(float2);
    if (smem > 48 * 1024) HOS_REFUSE("rotate_rows: %d rotated numbers do not fit", rot_dims);
    launch_pdl(rotate_rows_kernel, dim3(N), dim3(256), smem, stream, x, ld, Hq, Hk, dim, rot_dims, style, freq, token_pos,
               token_seq, k_mult);
    return check_launch("rotate_rows");
}

// keep_here: 1 only where every sequence of the step brings exactly one token: the kept inputs then move on inside this
// launch and hos_conv_keep is not needed.
// act: float32 [N][2 Gk dim + H vdim] (q, k, v after convolution, activation and lengths); beta_out, g_out: [N][H].
extern "C" int hos_conv_prep(const float* raw, long long ld, const float* conv_w, int taps, const float* conv_state,
                             const float* a_log, const float* dt_bias, const int* token_pos, const int* token_seq,
                             const int* cu_seqlens, const int* seq_slot, float* act, float* beta_out, float* g_out, int N,
                             int H, int Gk, int dim, int vdim, int keep_here, cudaStream_t stream) {
    if (N <= 0) return 0;
    if (taps < 1 || taps > kMaxTaps) HOS_REFUSE("conv_prep: %d taps are outside 1..%d", taps, kMaxTaps);
    const size_t smem = (size_t)2 * Gk * dim * sizeof(float);
    if (smem > 160 * 1024) HOS_REFUSE("conv_prep: %d query and key channels do not fit", 2 * Gk * dim);
    if (smem > 48 * 1024) cudaFuncSetAttribute(conv_prep_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    launch_pdl(conv_prep_kernel, dim3(N), dim3(256), smem, stream, raw, ld, conv_w, taps, conv_state, a_log, dt_bias,
               token_pos, token_seq, cu_seqlens, seq_slot, act, beta_out, g_out, H, Gk, dim, vdim,
               keep_here ? const_cast<float*>(conv_state) : (float*)nullptr);
    return check_launch("conv_prep");
}

extern "C" int hos_conv_keep(const float* raw, long long ld, const float* in_bias, int taps, float* conv_state, const int* token_pos,
                             const int* token_seq, const int* cu_seqlens, const int* seq_slot, int n_seqs, int C,
                             cudaStream_t stream) {
    if (n_seqs <= 0 || taps <= 1) return 0;
    if (taps > kMaxTaps) HOS_REFUSE("conv_keep: %d taps are outside 1..%d", taps, kMaxTaps);
    launch_pdl(short_conv_keep_kernel, dim3((C + 127) / 128, n_seqs), dim3(128), 0, stream, raw, ld, in_bias, taps, conv_state,
               token_pos, token_seq, cu_seqlens, seq_slot, C);
    return check_launch("conv_keep");
}

// raw: the rows from the first convolved column on, ld apart; w: [taps][C]; in_bias ([C] or null): added before the
// convolution; bias ([C] or null): after it; act: 0 none, 1 x logistic(x); conv_state: [slots][taps - 1][C]; out: float32
// [N][C].  single: 1 where every sequence of the step brings exactly one token: the kept inputs then move on inside this
// launch (otherwise hos_conv_keep does it afterwards).  dt_raw (or null): the rows from the first step-size column on, H of
// them, ld apart: dt_out [N][H] = softplus(dt_raw + dt_bias), g_out [N][H] = exp(-exp(a_log) dt).
extern "C" int hos_conv_act_rows(const float* raw, long long ld, const float* w, const float* in_bias, const float* bias, int taps,
                                 float* conv_state, int act, const int* token_pos, const int* token_seq, const int* cu_seqlens,
                                 const int* seq_slot, float* out, int N, int C, int single, const float* dt_raw, const float* dt_bias,
                                 const float* a_log, float* dt_out, float* g_out, int H, cudaStream_t stream) {
    if (N <= 0 || C <= 0) return 0;
    if (taps < 1 || taps > kMaxTaps) HOS_REFUSE("conv_act_rows: %d taps are outside 1..%d", taps, kMaxTaps);
    if (act != 0 && act != 1) HOS_REFUSE("conv_act_rows: unknown activation %d", act);
    if (dt_raw != nullptr && (dt_bias == nullptr || a_log == nullptr || dt_out == nullptr || g_out == nullptr || H <= 0))
        HOS_REFUSE("conv_act_rows: step sizes need their bias, their rates and two outputs");
    const bool vec = taps >= 2 && taps <= 4 && C % 4 == 0 && ld % 4 == 0 &&
                     (((uintptr_t)raw | (uintptr_t)out | (uintptr_t)conv_state | (uintptr_t)w | (uintptr_t)in_bias) % 16) == 0;
    const int per_block = 128 * (vec ? 4 : 1);
    const int conv_blocks = (C + per_block - 1) / per_block;
    const int run = conv_run(N, conv_blocks, single != 0);
    const dim3 grid(conv_blocks + (dt_raw != nullptr ? 1 : 0), (N + run - 1) / run);
    if (grid.y > 65535) HOS_REFUSE("conv_act_rows: %d rows are more than one launch takes", N);
    const ConvWalk c{raw, ld, w, in_bias, conv_state, single && taps > 1 ? conv_state : nullptr, token_pos, token_seq, cu_seqlens,
                     seq_slot, taps, C};
#define HOS_CAR(T, V)                                                                                                \
    launch_pdl(conv_act_rows_kernel<T, V>, grid, dim3(128), 0, stream, c, bias, act, out, N, run, conv_blocks, dt_raw, dt_bias, \
               a_log, dt_out, g_out, H)
#define HOS_CAR_V(T)                                                                                                 \
    do {                                                                                                             \
        if (vec) HOS_CAR(T, 4);                                                                                      \
        else HOS_CAR(T, 1);                                                                                          \
    } while (0)
    if (taps == 2) HOS_CAR_V(2);
    else if (taps == 3) HOS_CAR_V(3);
    else if (taps == 4) HOS_CAR_V(4);
    else HOS_CAR(0, 1);
#undef HOS_CAR_V
#undef HOS_CAR
    return check_launch("conv_act_rows");
}

// low: the rows' low-rank numbers from column 0 of `low` on, ld apart; w: [rank][C] (transposed), b: [C]; out: float32 [N][C].
extern "C" int hos_channel_decay(const float* low, long long ld, const float* w, const float* b, int rank, float tau, float* out,
                                 int N, int C, cudaStream_t stream) {
    if (N <= 0 || C <= 0) return 0;
    if (rank <= 0 || rank > 1024 || !(tau > 0.f)) HOS_REFUSE("channel_decay: a rank of %d and tau %g", rank, tau);
    const dim3 grid((C + 127) / 128, (N + kDecayRows - 1) / kDecayRows);
    if (grid.y > 65535) HOS_REFUSE("channel_decay: %d rows are more than one launch takes", N);
    launch_pdl(channel_decay_kernel, grid, dim3(128), (size_t)kDecayRows * rank * sizeof(float), stream, low, ld, w, b, rank,
               1.f / tau, out, N, C);
    return check_launch("channel_decay");
}
