// Several residual streams instead of one, and a norm without statistics.
//
// stream_mix_norm: the 32-bit residual h is [N, streams, width].  With y the sum of the parts of a
// sublayer's output (`delta`), every stream becomes
//     x_t <- sum_s mix[s, t] x_s + out_coef[t] * y,      all at once from the old streams,
// and what the next sublayer reads is
//     u = sum_t read[t] x_t   (the new streams; `read` null: their plain sum),
// normalised in one of two ways: tanh(alpha * u) * w + b (`alpha` given: no mean, no variance, nothing
// that ties a row's entries together), or u / rms(u) * w.  `mix` null: the streams keep their values;
// `out_coef` null: ones.  `delta` null: the streams stay as they are and are only read.  `rows` selects
// rows and leaves h alone; `out` null: only the streams are brought up to date.  One stream with
// nothing given but alpha is a plain residual with that norm.
//
// All sums are 32-bit and run in a fixed order: a stream's terms by rising s, then the output's; the
// reading by rising t.  With the tanh norm a row's entries are independent, so a row is cut among
// as many blocks as its width fills; the rms norm takes a block per row.
#include "common.cuh"
#include <math.h>

namespace {
constexpr int THREADS = 256;

__device__ __forceinline__ float block_sum(float v, float* red) {
    v = warp_sum(v);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float total = 0.f;
#pragma unroll
    for (int w = 0; w < THREADS / 32; ++w) total += red[w];
    return total;
}

template <int VEC>
struct Pack { float v[VEC]; };
template <int VEC>
__device__ __forceinline__ Pack<VEC> load_pack(const float* p) {
    Pack<VEC> r;
    if constexpr (VEC == 4) {
        float4 t = *reinterpret_cast<const float4*>(p);
        r.v[0] = t.x; r.v[1] = t.y; r.v[2] = t.z; r.v[3] = t.w;
    } else {
        r.v[0] = *p;
    }
    return r;
}
template <int VEC>
__device__ __forceinline__ void store_pack(float* p, const Pack<VEC>& r) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else *p = r.v[0];
}
template <int VEC>
__device__ __forceinline__ void store_pack(__nv_bfloat16* p, const Pack<VEC>& r) {
    if constexpr (VEC == 4) {
        __nv_bfloat162 lo = __floats2bfloat162_rn(r.v[0], r.v[1]), hi = __floats2bfloat162_rn(r.v[2], r.v[3]);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<unsigned*>(&lo), *reinterpret_cast<unsigned*>(&hi));
    } else {
        *p = __float2bfloat16_rn(r.v[0]);
    }
}

// grid: (rows, pieces of a row).  S: the most streams the instance holds in registers.
template <typename OutT, int VEC, int S, bool RMS>
__global__ void __launch_bounds__(THREADS)
stream_mix_norm_kernel(float* __restrict__ h, int streams, const float* __restrict__ delta, int num_partials,
                       size_t partial_stride, const float* __restrict__ mix, const float* __restrict__ out_coef,
                       const float* __restrict__ read, const float* __restrict__ weight,
                       const float* __restrict__ bias, const float* __restrict__ alpha, float eps,
                       OutT* __restrict__ out, const int* __restrict__ rows, int width) {
    extern __shared__ __align__(16) float row_buf[];  // [width], the rms norm's
    __shared__ float red[THREADS / 32];
    __shared__ float s_mix[S * S], s_out[S], s_read[S];
    ie_pdl_trigger();
    // (the coefficients are weights: no earlier kernel writes them)
    for (int i = threadIdx.x; i < S * S; i += THREADS) {
        int from = i / S, to = i - from * S;
        float c = from == to ? 1.f : 0.f;
        if (mix != nullptr) c = (from < streams && to < streams) ? mix[from * streams + to] : 0.f;
        s_mix[i] = c;
    }
    if (threadIdx.x < S) {
        bool there = threadIdx.x < streams;
        s_out[threadIdx.x] = !there ? 0.f : out_coef != nullptr ? out_coef[threadIdx.x] : 1.f;
        s_read[threadIdx.x] = !there ? 0.f : read != nullptr ? read[threadIdx.x] : 1.f;
    }
    float a = alpha != nullptr ? *alpha : 0.f;
    ie_pdl_wait();
    __syncthreads();
    size_t r = blockIdx.x, src = rows != nullptr ? (size_t)rows[r] : r;
    float* x_row = h + src * streams * width;
    const bool writes = delta != nullptr && rows == nullptr;
    float ss = 0.f;
    for (int i = (blockIdx.y * THREADS + threadIdx.x) * VEC; i < width; i += gridDim.y * THREADS * VEC) {
        Pack<VEC> x[S];
#pragma unroll
        for (int s = 0; s < S; ++s)
            if (s < streams) x[s] = load_pack<VEC>(x_row + (size_t)s * width + i);
        Pack<VEC> u;
#pragma unroll
        for (int v = 0; v < VEC; ++v) u.v[v] = 0.f;
        if (delta != nullptr) {
            Pack<VEC> y = load_pack<VEC>(delta + src * width + i);
#pragma unroll 4
            for (int p = 1; p < num_partials; ++p) {
                Pack<VEC> d = load_pack<VEC>(delta + p * partial_stride + src * width + i);
#pragma unroll
                for (int v = 0; v < VEC; ++v) y.v[v] += d.v[v];
            }
#pragma unroll
            for (int t = 0; t < S; ++t) {
                if (t >= streams) break;
                Pack<VEC> n;
#pragma unroll
                for (int v = 0; v < VEC; ++v) n.v[v] = 0.f;
#pragma unroll
                for (int s = 0; s < S; ++s) {
                    if (s >= streams) break;
                    float c = s_mix[s * S + t];
#pragma unroll
                    for (int v = 0; v < VEC; ++v) n.v[v] = fmaf(c, x[s].v[v], n.v[v]);
                }
                float o = s_out[t], rd = s_read[t];
#pragma unroll
                for (int v = 0; v < VEC; ++v) {
                    n.v[v] = fmaf(o, y.v[v], n.v[v]);
                    u.v[v] = fmaf(rd, n.v[v], u.v[v]);
                }
                if (writes) store_pack<VEC>(x_row + (size_t)t * width + i, n);
            }
        } else {
#pragma unroll
            for (int t = 0; t < S; ++t) {
                if (t >= streams) break;
                float rd = s_read[t];
#pragma unroll
                for (int v = 0; v < VEC; ++v) u.v[v] = fmaf(rd, x[t].v[v], u.v[v]);
            }
        }
        if (out == nullptr) continue;
        if constexpr (RMS) {
            store_pack<VEC>(row_buf + i, u);
#pragma unroll
            for (int v = 0; v < VEC; ++v) ss = fmaf(u.v[v], u.v[v], ss);
        } else {
            Pack<VEC> w = load_pack<VEC>(weight + i), b = load_pack<VEC>(bias + i);
#pragma unroll
            for (int v = 0; v < VEC; ++v) u.v[v] = fmaf(tanhf(a * u.v[v]), w.v[v], b.v[v]);
            store_pack<VEC>(out + r * width + i, u);
        }
    }
    if constexpr (RMS) {
        if (out == nullptr) return;
        float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)width + eps);
        for (int i = threadIdx.x * VEC; i < width; i += THREADS * VEC) {  // (a thread reads what it wrote)
            Pack<VEC> u = load_pack<VEC>(row_buf + i), w = load_pack<VEC>(weight + i);
#pragma unroll
            for (int v = 0; v < VEC; ++v) u.v[v] = w.v[v] * (u.v[v] * inv);
            store_pack<VEC>(out + r * width + i, u);
        }
    }
}

struct Args {
    float* h; int streams; const float* delta; int num_partials; size_t partial_stride;
    const float *mix, *out_coef, *read, *weight, *bias, *alpha; float eps; void* out; const int* rows;
    int num_rows, width; cudaStream_t stream;
};

template <typename OutT, int VEC, int S>
int launch(const Args& p) {
    const bool rms = p.alpha == nullptr && p.out != nullptr;
    if (rms) {
        size_t smem = (size_t)p.width * sizeof(float);
        if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
        static IePerDevice allowed;
        cudaError_t e = ie_allow_smem(allowed, stream_mix_norm_kernel<OutT, VEC, S, true>, 200 * 1024);
        if (e != cudaSuccess) return (int)e;
        return ie_launch(stream_mix_norm_kernel<OutT, VEC, S, true>, dim3(p.num_rows), dim3(THREADS), smem, p.stream,
                         p.h, p.streams, p.delta, p.num_partials, p.partial_stride, p.mix, p.out_coef, p.read,
                         p.weight, p.bias, p.alpha, p.eps, (OutT*)p.out, p.rows, p.width);
    }
    dim3 grid(p.num_rows, (p.width + THREADS * VEC - 1) / (THREADS * VEC));
    return ie_launch(stream_mix_norm_kernel<OutT, VEC, S, false>, grid, dim3(THREADS), 0, p.stream, p.h, p.streams,
                     p.delta, p.num_partials, p.partial_stride, p.mix, p.out_coef, p.read, p.weight, p.bias, p.alpha,
                     p.eps, (OutT*)p.out, p.rows, p.width);
}
template <typename OutT, int VEC>
int pick(const Args& p) {
    if (p.streams == 1) return launch<OutT, VEC, 1>(p);
    if (p.streams == 2) return launch<OutT, VEC, 2>(p);
    if (p.streams <= 4) return launch<OutT, VEC, 4>(p);
    return launch<OutT, 1, 16>(p);  // (so many streams in registers: one entry of a row per thread)
}
}  // namespace

// weight, bias: [width] (the bias with the tanh norm only); alpha: one number on the device, or null for
// the rms norm.
IE_API int ie_stream_mix_norm(float* h, int streams, const float* delta, int num_partials, long long partial_stride,
                              const float* mix, const float* out_coef, const float* read, const float* weight,
                              const float* bias, const float* alpha, float eps, void* out, int out_dtype,
                              const int* rows, int num_rows, int width, void* stream) {
    if (num_rows <= 0 || width <= 0) return 0;
    if (streams < 1 || streams > 16 || (delta != nullptr && num_partials < 1)) return (int)cudaErrorInvalidValue;
    if (out != nullptr && (weight == nullptr || (alpha != nullptr && bias == nullptr))) return (int)cudaErrorInvalidValue;
    Args p{h, streams, delta, num_partials, (size_t)partial_stride, mix, out_coef, read, weight, bias, alpha, eps, out,
           rows, num_rows, width, (cudaStream_t)stream};
    bool vec = width % 4 == 0 && (size_t)partial_stride % 4 == 0 &&
               ((reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(delta) |
                 reinterpret_cast<uintptr_t>(weight) | reinterpret_cast<uintptr_t>(bias) |
                 reinterpret_cast<uintptr_t>(out)) % 16 == 0);
    if (out_dtype == IE_BF16) return vec ? pick<__nv_bfloat16, 4>(p) : pick<__nv_bfloat16, 1>(p);
    return vec ? pick<float, 4>(p) : pick<float, 1>(p);
}
