// Hyper-connections: the residual stream is S copies ("streams") of the width, x [N][S][D] in 32-bit.  A branch reads a
// weighted sum of the streams, and its output goes back to all of them while they are mixed:
//   u = sum_s in[s] x_s;  y = branch(norm(u));  x_t <- sum_s mix[s][t] x_s + out[t] y      (all t at once, from the old x)
//
// hyper_norm: the update with a branch's output and what the NEXT branch reads, in one launch:
//   x_t <- sum_s mix[s][t] x_s + out[t] (y + bias);  h = RMSNorm(sum_s in_next[s] x_s; w, eps)
//   y: rows of either type, or 32-bit partial sums [parts][N][D] of a product that split K, added here in a fixed order;
//   without y the streams are left as they are; without in_next the weights are ones (the model's last norm reads the
//   sum of the streams).  A block per row: the streams' numbers of a column are in registers, the weighted sum is kept in
//   shared memory between the two passes.
// stream_sums: out = sum_s x_s of chosen rows (or all), 32-bit.
#include "common.cuh"

namespace hos {

constexpr int kMaxStreams = 16;

template <int VEC> struct Pack { float v[VEC]; };

template <int VEC>
__device__ __forceinline__ Pack<VEC> ld_pack(const float* p) {
    Pack<VEC> r;
    if constexpr (VEC == 4) {
        const float4 t = *(const float4*)p;
        r.v[0] = t.x; r.v[1] = t.y; r.v[2] = t.z; r.v[3] = t.w;
    } else {
        r.v[0] = *p;
    }
    return r;
}
template <int VEC>
__device__ __forceinline__ Pack<VEC> ld_pack(const bf16* p) {
    Pack<VEC> r;
    if constexpr (VEC == 4) {
        const uint2 u = *(const uint2*)p;
        r.v[0] = __uint_as_float(u.x << 16); r.v[1] = __uint_as_float(u.x & 0xffff0000u);
        r.v[2] = __uint_as_float(u.y << 16); r.v[3] = __uint_as_float(u.y & 0xffff0000u);
    } else {
        r.v[0] = to_float(*p);
    }
    return r;
}
template <int VEC>
__device__ __forceinline__ void st_pack(float* p, const Pack<VEC>& r) {
    if constexpr (VEC == 4) *(float4*)p = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else *p = r.v[0];
}
template <int VEC>
__device__ __forceinline__ void st_pack(bf16* p, const Pack<VEC>& r) {
    if constexpr (VEC == 4) {
        __nv_bfloat162 a = __floats2bfloat162_rn(r.v[0], r.v[1]), b = __floats2bfloat162_rn(r.v[2], r.v[3]);
        *(uint2*)p = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
    } else {
        *p = from_float<bf16>(r.v[0]);
    }
}

// SMAX: how many streams' numbers a thread holds; S of them are there (S == SMAX up to four).
template <int SMAX, int VEC>
__global__ void __launch_bounds__(512)
hyper_norm_kernel(const void* __restrict__ y, int y_bf16, int n_parts, long long part_stride, const float* __restrict__ bias,
                  float* __restrict__ x, int S_rt, const float* __restrict__ mix, const float* __restrict__ out_w,
                  const float* __restrict__ in_next, const float* __restrict__ w, float eps, void* __restrict__ h, int h_bf16,
                  int D) {
    pdl_enter();
    extern __shared__ float row[];               // [D] the weighted sum
    __shared__ float scratch[32];
    __shared__ float cs[kMaxStreams * kMaxStreams + 2 * kMaxStreams];      // mix, out, in_next
    const int S = SMAX <= 4 ? SMAX : S_rt;
    float* mix_s = cs;
    float* out_s = cs + S * S;
    float* in_s = out_s + S;
    for (int i = threadIdx.x; i < S * S; i += blockDim.x) mix_s[i] = y != nullptr ? mix[i] : 0.f;
    for (int i = threadIdx.x; i < S; i += blockDim.x) {
        out_s[i] = y != nullptr ? out_w[i] : 0.f;
        in_s[i] = in_next != nullptr ? in_next[i] : 1.f;
    }
    __syncthreads();
    const size_t n = blockIdx.x;
    float* xr = x + n * (size_t)S * D;
    float ss = 0.f;
    for (int d = threadIdx.x * VEC; d < D; d += blockDim.x * VEC) {
        Pack<VEC> old[SMAX];
#pragma unroll
        for (int s = 0; s < SMAX; ++s)
            if (s < S) old[s] = ld_pack<VEC>(xr + (size_t)s * D + d);
        Pack<VEC> u;
#pragma unroll
        for (int i = 0; i < VEC; ++i) u.v[i] = 0.f;
        if (y != nullptr) {
            Pack<VEC> b;
            if (y_bf16) {
                b = ld_pack<VEC>((const bf16*)y + n * D + d);
            } else {
                b = ld_pack<VEC>((const float*)y + n * D + d);
                for (int p = 1; p < n_parts; ++p) {
                    const Pack<VEC> c = ld_pack<VEC>((const float*)y + (size_t)p * part_stride + n * D + d);
#pragma unroll
                    for (int i = 0; i < VEC; ++i) b.v[i] += c.v[i];
                }
            }
            if (bias != nullptr) {
                const Pack<VEC> c = ld_pack<VEC>(bias + d);
#pragma unroll
                for (int i = 0; i < VEC; ++i) b.v[i] += c.v[i];
            }
#pragma unroll
            for (int t = 0; t < SMAX; ++t) {
                if (t >= S) break;
                Pack<VEC> nx;
#pragma unroll
                for (int i = 0; i < VEC; ++i) nx.v[i] = out_s[t] * b.v[i];
#pragma unroll
                for (int s = 0; s < SMAX; ++s) {
                    if (s >= S) break;
                    const float m = mix_s[s * S + t];
#pragma unroll
                    for (int i = 0; i < VEC; ++i) nx.v[i] = fmaf(m, old[s].v[i], nx.v[i]);
                }
                st_pack<VEC>(xr + (size_t)t * D + d, nx);
#pragma unroll
                for (int i = 0; i < VEC; ++i) u.v[i] = fmaf(in_s[t], nx.v[i], u.v[i]);
            }
        } else {
#pragma unroll
            for (int s = 0; s < SMAX; ++s) {
                if (s >= S) break;
#pragma unroll
                for (int i = 0; i < VEC; ++i) u.v[i] = fmaf(in_s[s], old[s].v[i], u.v[i]);
            }
        }
        if (h != nullptr) {
#pragma unroll
            for (int i = 0; i < VEC; ++i) ss = fmaf(u.v[i], u.v[i], ss);
            st_pack<VEC>(row + d, u);
        }
    }
    if (h == nullptr) return;
    ss = block_sum(ss, scratch);
    const float inv = 1.f / sqrtf(ss / (float)D + eps);
    for (int d = threadIdx.x * VEC; d < D; d += blockDim.x * VEC) {       // every thread reads back what it wrote
        Pack<VEC> u = ld_pack<VEC>(row + d);
        const Pack<VEC> wv = ld_pack<VEC>(w + d);
#pragma unroll
        for (int i = 0; i < VEC; ++i) u.v[i] = u.v[i] * inv * wv.v[i];
        if (h_bf16) st_pack<VEC>((bf16*)h + n * D + d, u);
        else st_pack<VEC>((float*)h + n * D + d, u);
    }
}

__global__ void stream_sums_kernel(const float* __restrict__ x, const int* __restrict__ rows, float* __restrict__ out, int S, int D) {
    pdl_enter();
    const size_t src = rows != nullptr ? (size_t)rows[blockIdx.x] : (size_t)blockIdx.x;
    for (int d = threadIdx.x; d < D; d += blockDim.x) {
        float v = 0.f;
        for (int s = 0; s < S; ++s) v += x[(src * S + s) * D + d];
        out[(size_t)blockIdx.x * D + d] = v;
    }
}

}  // namespace hos

using namespace hos;

// x: float32 [N][S][D].  y (or null: no update): [N][D] of y_dtype, or n_parts > 1 planes of float32 partial sums; bias: [D]
// float32 added to y, or null; mix: [S][S] as [from][to]; out_w: [S]; in_next: [S] or null (ones); h (of h_dtype, or null): the
// RMS norm with weight w of the weighted sum of the new streams.
extern "C" int hos_hyper_norm(const void* y, int y_dtype, int n_parts, const float* bias, float* x, int S, const float* mix,
                              const float* out_w, const float* in_next, const float* w, float eps, void* h, int h_dtype, int N, int D,
                              cudaStream_t stream) {
    if (N <= 0) return 0;
    if (S < 1 || S > kMaxStreams) HOS_REFUSE("hyper_norm: %d streams are outside 1..%d", S, kMaxStreams);
    if (y != nullptr && (mix == nullptr || out_w == nullptr)) HOS_REFUSE("hyper_norm: a branch's output needs the mixing weights");
    if (h != nullptr && w == nullptr) HOS_REFUSE("hyper_norm: a norm needs its weight");
    if (n_parts > 1 && y_dtype != kF32) HOS_REFUSE("hyper_norm: partial sums must be float32");
    const size_t smem = (size_t)D * sizeof(float);
    if (smem > 200 * 1024) HOS_REFUSE("hyper_norm: width %d does not fit a block's shared memory", D);
    const bool vec = D % 4 == 0 && (uintptr_t)y % 16 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)h % 16 == 0 &&
                     (uintptr_t)bias % 16 == 0 && (uintptr_t)w % 16 == 0;
    // few rows: as many threads as there are columns to take (a row is one block's chain); many rows: 256
    int threads = 128;
    const int most = N <= 2 * sm_count_cached() ? 512 : 256;
    while (threads < most && threads * (vec ? 4 : 1) < D) threads *= 2;
    const long long plane = (long long)N * D;
#define HOS_HN(SM, V)                                                                                                \
    do {                                                                                                             \
        if (smem > 48 * 1024)                                                                                        \
            cudaFuncSetAttribute(hyper_norm_kernel<SM, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);  \
        launch_pdl(hyper_norm_kernel<SM, V>, dim3(N), dim3(threads), smem, stream, y, y_dtype == kBF16 ? 1 : 0, n_parts, plane, \
                   bias, x, S, mix, out_w, in_next, w, eps, h, h_dtype == kBF16 ? 1 : 0, D);                         \
    } while (0)
#define HOS_HN_V(SM)                                                                                                 \
    do {                                                                                                             \
        if (vec) HOS_HN(SM, 4);                                                                                      \
        else HOS_HN(SM, 1);                                                                                          \
    } while (0)
    if (S == 1) HOS_HN_V(1);
    else if (S == 2) HOS_HN_V(2);
    else if (S == 3) HOS_HN_V(3);
    else if (S == 4) HOS_HN_V(4);
    else HOS_HN(16, 1);
#undef HOS_HN_V
#undef HOS_HN
    return check_launch("hyper_norm");
}

// out[i] = the sum of the S streams of row rows[i] of x (rows null: row i), float32 [n][D].
extern "C" int hos_stream_sums(const float* x, const int* rows, float* out, int n, int S, int D, cudaStream_t stream) {
    if (n <= 0) return 0;
    launch_pdl(stream_sums_kernel, dim3(n), dim3(256), 0, stream, x, rows, out, S, D);
    return check_launch("stream_sums");
}
