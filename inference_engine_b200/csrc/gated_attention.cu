// Input stage of an attention whose queries and keys are normalised per head before the rotation,
// and whose value rows may have another size than its key rows.  Variants by parameters: a bias on
// the whole projection (`bias`, laid out like a row of it, added first); no norm on queries or keys
// (their weight is null); value heads divided by their root mean square over `vdim` (eps inside the
// root, no weight) before they are cached (`value_norm`); values that are the keys as projected
// (with their bias, before norm and rotation: `values_from_keys`; the projection then holds no value
// columns and vdim = dim); queries and keys divided by their root mean square without a weight
// (`unit_norm`); query heads multiplied by a number per head (`q_head_scale`) and by
// 1 + warm_coef * ln(floor((p + 1) / warm_every) + 1) at position p (`warm_every` > 0); the rotation's pairs (`interleaved` 0: entry i with entry i + rot_dims / 2;
// 1: entry 2i with entry 2i + 1; the table of angles is the same).
//
// qk_norm_rope_write: from the fused 32-bit projection [N, ld] = (heads * dim queries, kv_heads *
// dim keys, kv_heads * vdim values): every query and key head is divided by its root mean square
// over `dim` (eps inside the root) and multiplied by a weight of size `dim` that all heads share;
// the first rot_dims entries of the head are rotated by the token's position (entry i pairs with
// entry i + rot_dims / 2; cos and sin come from the 32-bit table [positions, 2, rot_dims / 2]);
// queries go to q_out [N, heads * dim], keys and values into the request's page rows
// (k_cache [pages, kv_heads, page_size, dim], v_cache [pages, kv_heads, page_size, vdim]).
// One warp per (token, head of q, k or v); the sums do not depend on the rest of the step.
//
// qk_wide_norm_rope_write: the same stage with one norm over all query columns of a token and one over all
// its key columns, before they are split into heads (weights as long as the columns).  A block per token.
// `value_scale` (both kernels) multiplies the values before they are cached, for a mixer whose output is
// wanted times a constant.
#include "common.cuh"
#include <math.h>

namespace {
constexpr int QW_WARPS = 4;

template <typename T>
__global__ void __launch_bounds__(QW_WARPS * 32)
qk_norm_rope_write_kernel(const float* __restrict__ proj, int ld, const int* __restrict__ positions,
                          const float* __restrict__ table, int rot_dims, int table_positions,
                          const float* __restrict__ bias, int value_norm, int values_from_keys, int interleaved,
                          const float* __restrict__ q_weight, const float* __restrict__ k_weight, float eps,
                          int unit_norm, const float* __restrict__ q_head_scale, float warm_coef, int warm_every,
                          float value_scale, T* __restrict__ q_out, T* __restrict__ k_cache, T* __restrict__ v_cache,
                          const int* __restrict__ slot_mapping, int heads, int kv_heads, int dim, int vdim,
                          int page_size, int total_pages, int* err) {
    extern __shared__ float rows[];  // [QW_WARPS][dim]
    ie_pdl_trigger();
    ie_pdl_wait();
    int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    int unit = blockIdx.y * QW_WARPS + warp;
    int n = blockIdx.x;
    int units = heads + 2 * kv_heads;
    if (unit >= units) return;
    const float* src = proj + (size_t)n * ld;
    long long cache_row = -1;
    if (unit >= heads) {
        if (slot_mapping == nullptr) return;  // a run that borrows another layer's cache writes nothing
        int slot = slot_mapping[n];
        int page = slot / page_size;
        if (slot < 0 || page >= total_pages) {
            if (lane == 0) ie_report(err, IE_ERR_PAGE, slot, n);
            return;
        }
        int g = (unit - heads) % kv_heads;
        cache_row = ((long long)page * kv_heads + g) * page_size + (slot % page_size);
    }
    if (unit >= heads + kv_heads) {  // a value head: copied as it is, or divided by its root mean square
        int g = unit - heads - kv_heads;
        size_t col = values_from_keys ? (size_t)(heads + g) * dim : (size_t)(heads + kv_heads) * dim + (size_t)g * vdim;
        const float* v = src + col;
        const float* vb = bias != nullptr ? bias + col : nullptr;
        float inv = value_scale;
        if (value_norm) {
            float ss = 0.f;
            for (int d = lane; d < vdim; d += 32) {
                float e = vb != nullptr ? v[d] + vb[d] : v[d];
                ss = fmaf(e, e, ss);
            }
            ss = warp_sum(ss);
            inv = value_scale / sqrtf(ss / (float)vdim + eps);
        }
        for (int d = lane; d < vdim; d += 32)
            ie_store(v_cache + cache_row * vdim + d, (vb != nullptr ? v[d] + vb[d] : v[d]) * inv);
        return;
    }
    bool is_q = unit < heads;
    const float* x = src + (size_t)unit * dim;  // (the key heads follow the query heads)
    const float* xb = bias != nullptr ? bias + (size_t)unit * dim : nullptr;
    const float* weight = is_q ? q_weight : k_weight;
    float* y = rows + warp * dim;
    float ss = 0.f;
    for (int d = lane; d < dim; d += 32) {
        float e = xb != nullptr ? x[d] + xb[d] : x[d];
        y[d] = e;
        ss = fmaf(e, e, ss);
    }
    ss = warp_sum(ss);
    float inv = 1.0f / sqrtf(ss / (float)dim + eps);
    if (weight != nullptr)
        for (int d = lane; d < dim; d += 32) y[d] = (y[d] * inv) * weight[d];
    __syncwarp();
    int pos = positions[n];
    float factor = (unit_norm && weight == nullptr) ? inv : 1.0f;
    if (is_q) {
        if (q_head_scale != nullptr) factor *= q_head_scale[unit];
        if (warm_every > 0) factor *= 1.0f + warm_coef * logf((float)((pos + 1) / warm_every + 1));
    }
    int half = rot_dims / 2;
    if (half > 0 && (pos < 0 || pos >= table_positions)) {
        if (lane == 0) ie_report(err, IE_ERR_POSITION, pos, n);
        return;
    }
    T* dst = is_q ? q_out + ((size_t)n * heads + unit) * dim : k_cache + cache_row * dim;
    for (int d = lane; d < dim; d += 32) {
        float r = y[d];
        if (interleaved) {
            if (d < rot_dims) {
                int j = d >> 1;
                float c = table[((size_t)pos * 2) * half + j], s = table[((size_t)pos * 2 + 1) * half + j];
                r = (d & 1) ? y[d] * c + y[d - 1] * s : y[d] * c - y[d + 1] * s;
            }
        } else if (d < half) {
            float c = table[((size_t)pos * 2) * half + d], s = table[((size_t)pos * 2 + 1) * half + d];
            r = y[d] * c - y[d + half] * s;
        } else if (d < rot_dims) {
            float c = table[((size_t)pos * 2) * half + (d - half)], s = table[((size_t)pos * 2 + 1) * half + (d - half)];
            r = y[d] * c + y[d - half] * s;
        }
        ie_store(dst + d, r * factor);
    }
}

constexpr int WN_THREADS = 256;

__device__ __forceinline__ float wide_sum(float v, float* red) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float total = 0.f;
#pragma unroll
    for (int w = 0; w < WN_THREADS / 32; ++w) total += red[w];
    return total;
}

template <typename T>
__global__ void __launch_bounds__(WN_THREADS)
qk_wide_norm_rope_write_kernel(const float* __restrict__ proj, int ld, const int* __restrict__ positions,
                               const float* __restrict__ table, int rot_dims, int table_positions,
                               const float* __restrict__ bias, int interleaved, const float* __restrict__ q_weight,
                               const float* __restrict__ k_weight, float eps, float value_scale, T* __restrict__ q_out,
                               T* __restrict__ k_cache, T* __restrict__ v_cache, const int* __restrict__ slot_mapping,
                               int heads, int kv_heads, int dim, int vdim, int page_size, int total_pages, int* err) {
    extern __shared__ float row[];  // the token's query columns, then its key columns
    __shared__ float red_q[WN_THREADS / 32], red_k[WN_THREADS / 32];
    ie_pdl_trigger();
    ie_pdl_wait();
    const int n = blockIdx.x, tid = threadIdx.x, nq = heads * dim, nqk = (heads + kv_heads) * dim;
    const float* src = proj + (size_t)n * ld;
    float sq = 0.f, sk = 0.f;
    for (int i = tid; i < nqk; i += WN_THREADS) {
        float e = bias != nullptr ? src[i] + bias[i] : src[i];
        row[i] = e;
        if (i < nq) sq = fmaf(e, e, sq);
        else sk = fmaf(e, e, sk);
    }
    const float inv_q = 1.0f / sqrtf(wide_sum(sq, red_q) / (float)nq + eps);
    const float inv_k = 1.0f / sqrtf(wide_sum(sk, red_k) / (float)(nqk - nq) + eps);
    for (int i = tid; i < nqk; i += WN_THREADS) row[i] = (row[i] * (i < nq ? inv_q : inv_k)) * (i < nq ? q_weight[i] : k_weight[i - nq]);
    __syncthreads();
    const int pos = positions[n], half = rot_dims / 2;
    if (half > 0 && (pos < 0 || pos >= table_positions)) {
        if (tid == 0) ie_report(err, IE_ERR_POSITION, pos, n);
        return;
    }
    int slot = slot_mapping != nullptr ? slot_mapping[n] : -1, page = slot / page_size;
    bool writes = slot_mapping != nullptr;
    if (writes && (slot < 0 || page >= total_pages)) {
        if (tid == 0) ie_report(err, IE_ERR_PAGE, slot, n);
        writes = false;
    }
    const float* cs = table + (size_t)max(pos, 0) * rot_dims;  // cos of the angles, then their sin
    const long long first_row = (long long)page * kv_heads * page_size + (slot - page * page_size);
    for (int i = tid; i < (writes ? nqk : nq); i += WN_THREADS) {
        int unit = i / dim, d = i - unit * dim;
        float r = row[i];
        if (d < rot_dims) {
            int j = interleaved ? d >> 1 : (d < half ? d : d - half);
            bool second = interleaved ? (d & 1) : d >= half;
            float c = cs[j], s = cs[half + j], other = row[interleaved ? (second ? i - 1 : i + 1) : (second ? i - half : i + half)];
            r = second ? r * c + other * s : r * c - other * s;
        }
        if (i < nq) ie_store(q_out + (size_t)n * nq + i, r);
        else ie_store(k_cache + (first_row + (long long)(unit - heads) * page_size) * dim + d, r);
    }
    if (!writes) return;
    for (int i = tid; i < kv_heads * vdim; i += WN_THREADS) {
        int g = i / vdim, d = i - g * vdim;
        float e = bias != nullptr ? src[nqk + i] + bias[nqk + i] : src[nqk + i];
        ie_store(v_cache + (first_row + (long long)g * page_size) * vdim + d, e * value_scale);
    }
}

// The same, four entries at a time (sizes and addresses allow it): a thread holds its pieces of the token's
// columns in registers; norm weights and biases, which no kernel writes, are asked for before the wait.
constexpr int WV_THREADS = 512, WV_PIECES = 4;

__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
    __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<unsigned*>(&lo), *reinterpret_cast<unsigned*>(&hi));
}

template <typename T>
__global__ void __launch_bounds__(WV_THREADS)
qk_wide_norm_rope_write4_kernel(const float* __restrict__ proj, int ld, const int* __restrict__ positions,
                                const float* __restrict__ table, int rot_dims, int table_positions,
                                const float* __restrict__ bias, int interleaved, const float* __restrict__ q_weight,
                                const float* __restrict__ k_weight, float eps, float value_scale, T* __restrict__ q_out,
                                T* __restrict__ k_cache, T* __restrict__ v_cache, const int* __restrict__ slot_mapping,
                                int heads, int kv_heads, int dim, int vdim, int page_size, int total_pages, int* err) {
    extern __shared__ __align__(16) float row[];  // halves: the normalised columns, for the pairs' other entries
    __shared__ float red[2][WV_THREADS / 32];
    ie_pdl_trigger();
    const int n = blockIdx.x, tid = threadIdx.x, nq = heads * dim, nqk = (heads + kv_heads) * dim, all = nqk + kv_heads * vdim;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    float4 w[WV_PIECES], e[WV_PIECES];
#pragma unroll
    for (int i = 0; i < WV_PIECES; ++i) {
        int c = (i * WV_THREADS + tid) * 4;
        w[i] = c < nq ? *reinterpret_cast<const float4*>(q_weight + c)
             : c < nqk ? *reinterpret_cast<const float4*>(k_weight + c - nq) : zero;
        e[i] = c < all && bias != nullptr ? *reinterpret_cast<const float4*>(bias + c) : zero;
    }
    ie_pdl_wait();
    const float* src = proj + (size_t)n * ld;
    const int pos = positions[n], half = rot_dims / 2;
    const int slot = slot_mapping != nullptr ? slot_mapping[n] : -1;
    float sq = 0.f, sk = 0.f;
#pragma unroll
    for (int i = 0; i < WV_PIECES; ++i) {
        int c = (i * WV_THREADS + tid) * 4;
        if (c >= all) break;
        float4 x = *reinterpret_cast<const float4*>(src + c);
        e[i].x += x.x; e[i].y += x.y; e[i].z += x.z; e[i].w += x.w;
    }
#pragma unroll
    for (int i = 0; i < WV_PIECES; ++i) {
        int c = (i * WV_THREADS + tid) * 4;
        float s = fmaf(e[i].x, e[i].x, fmaf(e[i].y, e[i].y, fmaf(e[i].z, e[i].z, e[i].w * e[i].w)));
        if (c < nq) sq += s;
        else if (c < nqk) sk += s;
    }
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if ((tid & 31) == 0) { red[0][tid >> 5] = sq; red[1][tid >> 5] = sk; }
    __syncthreads();
    sq = sk = 0.f;
#pragma unroll
    for (int i = 0; i < WV_THREADS / 32; ++i) { sq += red[0][i]; sk += red[1][i]; }
    const float inv_q = 1.0f / sqrtf(sq / (float)nq + eps), inv_k = 1.0f / sqrtf(sk / (float)(nqk - nq) + eps);
#pragma unroll
    for (int i = 0; i < WV_PIECES; ++i) {
        int c = (i * WV_THREADS + tid) * 4;
        if (c >= nqk) continue;
        float inv = c < nq ? inv_q : inv_k;
        e[i].x = (e[i].x * inv) * w[i].x; e[i].y = (e[i].y * inv) * w[i].y;
        e[i].z = (e[i].z * inv) * w[i].z; e[i].w = (e[i].w * inv) * w[i].w;
        if (!interleaved && rot_dims > 0) *reinterpret_cast<float4*>(row + c) = e[i];
    }
    if (half > 0 && (pos < 0 || pos >= table_positions)) {
        if (tid == 0) ie_report(err, IE_ERR_POSITION, pos, n);
        return;
    }
    int page = slot / page_size;
    bool writes = slot_mapping != nullptr;
    if (writes && (slot < 0 || page >= total_pages)) {
        if (tid == 0) ie_report(err, IE_ERR_PAGE, slot, n);
        writes = false;
    }
    if (!interleaved && rot_dims > 0) __syncthreads();
    const float* cs = table + (size_t)max(pos, 0) * rot_dims;  // cos of the angles, then their sin
    const long long first_row = (long long)page * kv_heads * page_size + (slot - page * page_size);
#pragma unroll
    for (int i = 0; i < WV_PIECES; ++i) {
        int c = (i * WV_THREADS + tid) * 4;
        if (c >= all || (c >= nq && !writes)) break;
        float4 x = e[i];
        if (c >= nqk) {
            int g = (c - nqk) / vdim, d = c - nqk - g * vdim;
            x.x *= value_scale; x.y *= value_scale; x.z *= value_scale; x.w *= value_scale;
            store4(v_cache + (first_row + (long long)g * page_size) * vdim + d, x);
            continue;
        }
        int unit = c / dim, d = c - unit * dim;
        if (d < rot_dims) {
            if (interleaved) {
                float2 co = *reinterpret_cast<const float2*>(cs + (d >> 1)), si = *reinterpret_cast<const float2*>(cs + half + (d >> 1));
                x = make_float4(x.x * co.x - x.y * si.x, x.y * co.x + x.x * si.x, x.z * co.y - x.w * si.y, x.w * co.y + x.z * si.y);
            } else {
                bool second = d >= half;
                int j = second ? d - half : d;
                float4 co = *reinterpret_cast<const float4*>(cs + j), si = *reinterpret_cast<const float4*>(cs + half + j);
                float4 o = *reinterpret_cast<const float4*>(row + (second ? c - half : c + half));
                float sg = second ? 1.f : -1.f;
                x = make_float4(x.x * co.x + sg * (o.x * si.x), x.y * co.y + sg * (o.y * si.y),
                                x.z * co.z + sg * (o.z * si.z), x.w * co.w + sg * (o.w * si.w));
            }
        }
        if (c < nq) store4(q_out + (size_t)n * nq + c, x);
        else store4(k_cache + (first_row + (long long)(unit - heads) * page_size) * dim + d, x);
    }
}
}  // namespace

IE_API int ie_qk_norm_rope_write(const float* proj, int ld, const int* positions, const float* table, int rot_dims,
                                 int table_positions, const float* bias, int value_norm, int values_from_keys,
                                 int interleaved, const float* q_weight,
                                 const float* k_weight, float eps, int unit_norm, const float* q_head_scale,
                                 float warm_coef, int warm_every, float value_scale, void* q_out, void* k_cache, void* v_cache, int dtype, const int* slot_mapping,
                                 int num_tokens, int heads, int kv_heads, int dim, int vdim, int page_size,
                                 int total_pages, int* err, void* stream) {
    if (num_tokens <= 0) return 0;
    if (rot_dims < 0 || rot_dims % 2 || rot_dims > dim || (rot_dims > 0 && table == nullptr))
        return (int)cudaErrorInvalidValue;
    if ((values_from_keys && vdim != dim) || warm_every < 0) return (int)cudaErrorInvalidValue;
    size_t smem = (size_t)QW_WARPS * dim * sizeof(float);
    if (smem > 48 * 1024) return (int)cudaErrorInvalidValue;
    int units = heads + 2 * kv_heads;
    dim3 grid(num_tokens, (units + QW_WARPS - 1) / QW_WARPS);
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == IE_BF16)
        return ie_launch(qk_norm_rope_write_kernel<__nv_bfloat16>, grid, dim3(QW_WARPS * 32), smem, s, proj, ld,
                         positions, table, rot_dims, table_positions, bias, value_norm, values_from_keys, interleaved, q_weight, k_weight, eps, unit_norm, q_head_scale, warm_coef, warm_every, value_scale, (__nv_bfloat16*)q_out,
                         (__nv_bfloat16*)k_cache, (__nv_bfloat16*)v_cache, slot_mapping, heads, kv_heads, dim, vdim,
                         page_size, total_pages, err);
    return ie_launch(qk_norm_rope_write_kernel<float>, grid, dim3(QW_WARPS * 32), smem, s, proj, ld, positions, table,
                     rot_dims, table_positions, bias, value_norm, values_from_keys, interleaved, q_weight, k_weight, eps, unit_norm, q_head_scale, warm_coef, warm_every, value_scale, (float*)q_out, (float*)k_cache,
                     (float*)v_cache, slot_mapping, heads, kv_heads, dim, vdim, page_size, total_pages, err);
}

IE_API int ie_qk_wide_norm_rope_write(const float* proj, int ld, const int* positions, const float* table, int rot_dims,
                                      int table_positions, const float* bias, int interleaved, const float* q_weight,
                                      const float* k_weight, float eps, float value_scale, void* q_out, void* k_cache,
                                      void* v_cache, int dtype, const int* slot_mapping, int num_tokens, int heads,
                                      int kv_heads, int dim, int vdim, int page_size, int total_pages, int* err,
                                      void* stream) {
    if (num_tokens <= 0) return 0;
    if (rot_dims < 0 || rot_dims % 2 || rot_dims > dim || (rot_dims > 0 && table == nullptr) || q_weight == nullptr ||
        k_weight == nullptr)
        return (int)cudaErrorInvalidValue;
    size_t smem = (size_t)(heads + kv_heads) * dim * sizeof(float);
    if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
    cudaStream_t s = (cudaStream_t)stream;
    // (which of the two kernels runs depends on the sizes and on how the arrays lie, not on the step)
    const int all = (heads + kv_heads) * dim + kv_heads * vdim;
    const uintptr_t bits = reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(table) | reinterpret_cast<uintptr_t>(bias) |
                           reinterpret_cast<uintptr_t>(q_weight) | reinterpret_cast<uintptr_t>(k_weight) |
                           reinterpret_cast<uintptr_t>(q_out) | reinterpret_cast<uintptr_t>(k_cache) | reinterpret_cast<uintptr_t>(v_cache);
    if (dim % 4 == 0 && vdim % 4 == 0 && ld % 4 == 0 && rot_dims % (interleaved ? 4 : 8) == 0 && bits % 16 == 0 &&
        all <= 4 * WV_THREADS * WV_PIECES && smem <= 40 * 1024) {
        size_t rows = interleaved ? 0 : smem;
        if (dtype == IE_BF16)
            return ie_launch(qk_wide_norm_rope_write4_kernel<__nv_bfloat16>, dim3(num_tokens), dim3(WV_THREADS), rows, s, proj,
                             ld, positions, table, rot_dims, table_positions, bias, interleaved, q_weight, k_weight, eps,
                             value_scale, (__nv_bfloat16*)q_out, (__nv_bfloat16*)k_cache, (__nv_bfloat16*)v_cache,
                             slot_mapping, heads, kv_heads, dim, vdim, page_size, total_pages, err);
        return ie_launch(qk_wide_norm_rope_write4_kernel<float>, dim3(num_tokens), dim3(WV_THREADS), rows, s, proj, ld,
                         positions, table, rot_dims, table_positions, bias, interleaved, q_weight, k_weight, eps,
                         value_scale, (float*)q_out, (float*)k_cache, (float*)v_cache, slot_mapping, heads, kv_heads, dim,
                         vdim, page_size, total_pages, err);
    }
#define IE_WN_LAUNCH(T)                                                                                              \
    do {                                                                                                             \
        static IePerDevice allowed;                                                                                  \
        if (smem > 40 * 1024) {                                                                                      \
            cudaError_t e = ie_allow_smem(allowed, qk_wide_norm_rope_write_kernel<T>, 200 * 1024);                   \
            if (e != cudaSuccess) return (int)e;                                                                     \
        }                                                                                                            \
        return ie_launch(qk_wide_norm_rope_write_kernel<T>, dim3(num_tokens), dim3(WN_THREADS), smem, s, proj, ld,   \
                         positions, table, rot_dims, table_positions, bias, interleaved, q_weight, k_weight, eps,    \
                         value_scale, (T*)q_out, (T*)k_cache, (T*)v_cache, slot_mapping, heads, kv_heads, dim, vdim, \
                         page_size, total_pages, err);                                                               \
    } while (0)
    if (dtype == IE_BF16) IE_WN_LAUNCH(__nv_bfloat16);
    IE_WN_LAUNCH(float);
#undef IE_WN_LAUNCH
}
