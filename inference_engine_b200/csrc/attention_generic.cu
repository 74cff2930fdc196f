// Paged attention for any mix of prompt portions and decoded tokens, any head size that is
// a multiple of 8 up to 256, any number of heads and groups, 32-bit or bfloat16 cache.
//
// One warp per (token, query head).  The query at absolute position p of its request sees
// the keys at positions lo .. p of the same request (lo = 0, or p - window + 1 with a
// window), found through the request's block table.  Keys are walked in tiles of 32 aligned
// to absolute position 0; scores, the running maximum, the running sum and the weighted sum
// of values are 32-bit, with the same order of operations whatever else is in the step: a
// position's result depends on its own request's data only.  This is the attention of the
// engine's 32-bit path, and the fallback of the bfloat16 path for head sizes its
// tensor-core kernels do not take.  Counterparts in the reference:
// engine/kernels/paged_attention.py:44-87 (decode rows) and the gather + SDPA path
// engine/model/layers.py:215-225 (prompt portions).
// A value row may be shorter than a key row and may live inside it: `hdv` entries at the start of
// rows `v_stride` apart (a mixer that caches one shared latent row per token passes the key cache
// as the value cache too, `v_stride` = the key row and `hdv` = the latent's size).
// `chunk` > 0: a query sees only the keys of its own chunk of that many positions (counted from the
// request's position 0).  `head_bias` != null: the weight of a visible key is sigmoid(score +
// head_bias[head]) and the weights are not normalised over the keys (no softmax).
// `sinks` != null (softmax only): the denominator holds one more term exp(sinks[head]) that has no
// key and no value; it is the state the running maximum and sum start from.  `out_gate` != null:
// the head's result is multiplied by sigmoid(out_gate[token * gate_ld + head]).
// `softcap` > 0: a score s (after the scale) becomes softcap * tanh(s / softcap).  `keep_first` > 0 (with
// a window): the keys at positions below `keep_first` stay visible to every later query of the request,
// beside its window; they keep their own positions.
// A bias by distance n = (query's position - key's position), added to the score after the scale:
// -log_r1[head] * ln(1 + log_r2[head] * n), and/or a table, bias_table[head * bias_len + min(n, bias_len -
// 1)].  Rows of the output lie `out_ld` entries apart.  `gate_elements` 1: `out_gate` holds a number per head and value entry ([token * gate_ld + head *
// hdv + d]) instead of one per head.
#include "common.cuh"
#include <math.h>

namespace {
constexpr int WARPS = 4;
constexpr int MAX_ACC = 16;  // value rows of up to 512 entries

template <typename T>
__device__ __forceinline__ float dot_row_any(const float* __restrict__ q, const T* __restrict__ k, int hd) {
    float s = 0.f;  // (rows that are not a multiple of 16 bytes: one entry at a time)
    for (int d = 0; d < hd; ++d) s = fmaf(q[d], ie_load(k + d), s);
    return s;
}
__device__ __forceinline__ float dot_row(const float* __restrict__ q, const float* __restrict__ k, int hd) {
    float s = 0.f;
    for (int d = 0; d < hd; d += 4) {
        float4 kv = *reinterpret_cast<const float4*>(k + d);
        s = fmaf(q[d], kv.x, s); s = fmaf(q[d + 1], kv.y, s);
        s = fmaf(q[d + 2], kv.z, s); s = fmaf(q[d + 3], kv.w, s);
    }
    return s;
}
__device__ __forceinline__ float dot_row(const float* __restrict__ q, const __nv_bfloat16* __restrict__ k, int hd) {
    float s = 0.f;
    for (int d = 0; d < hd; d += 8) {
        uint4 raw = *reinterpret_cast<const uint4*>(k + d);
        const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            float2 f = __bfloat1622float2(h2[i]);
            s = fmaf(q[d + 2 * i], f.x, s);
            s = fmaf(q[d + 2 * i + 1], f.y, s);
        }
    }
    return s;
}

template <typename T>
__global__ void __launch_bounds__(WARPS * 32)
paged_attention_generic_kernel(const T* __restrict__ q, const T* __restrict__ k_cache,
                               const T* __restrict__ v_cache, const int* __restrict__ block_tables,
                               int table_width, const int* __restrict__ seq_of_token,
                               const int* __restrict__ positions, T* __restrict__ out,
                               int nh, int nkv, int hd, int hdv, int v_stride, int page_size, int total_pages,
                               float scale, int window, int chunk, const float* __restrict__ head_bias,
                               const float* __restrict__ sinks, const float* __restrict__ out_gate, int gate_ld,
                               float softcap, int keep_first, int gate_elements, const float* __restrict__ log_r1,
                               const float* __restrict__ log_r2, const float* __restrict__ bias_table, int bias_len,
                               int out_ld, int* err) {
    extern __shared__ float q_smem[];  // [WARPS][hd]
    ie_pdl_trigger();
    ie_pdl_wait();
    int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    int head = blockIdx.x * WARPS + warp;
    int token = blockIdx.y;
    if (head >= nh) return;  // whole warp leaves together; no block-wide barrier below
    int kvh = head / (nh / nkv);
    int seq = seq_of_token[token], pos = positions[token];
    const int* table = block_tables + (size_t)seq * table_width;
    float* qs = q_smem + warp * hd;
    const T* qrow = q + ((size_t)token * nh + head) * hd;
    for (int d = lane; d < hd; d += 32) qs[d] = ie_load(qrow + d);
    __syncwarp();

    int lo = (window > 0 && pos - window + 1 > 0) ? pos - window + 1 : 0;
    if (chunk > 0) lo = max(lo, (pos / chunk) * chunk);  // chunks are counted from the request's position 0
    const int kept = min(keep_first, lo);  // keys below `kept` are seen beside the window's
    const float inv_cap = softcap > 0.f ? 1.0f / softcap : 0.f;
    const bool gated = head_bias != nullptr;  // sigmoid(score + bias) per key, not normalised over keys
    float hb = gated ? head_bias[head] : 0.f;
    float m = -INFINITY, l = 0.f;
    if (!gated && sinks != nullptr) { m = sinks[head]; l = 1.0f; }
    float acc[MAX_ACC];
#pragma unroll
    for (int i = 0; i < MAX_ACC; ++i) acc[i] = 0.f;
    int nacc = (hdv + 31) / 32;

    for (int t0 = kept > 0 ? 0 : (lo / 32) * 32; t0 <= pos; t0 += 32) {
        if (t0 >= kept && t0 + 31 < lo) {  // between the kept keys and the window: nothing to see
            t0 = (lo / 32) * 32 - 32;
            continue;
        }
        int kpos = t0 + lane;
        bool valid = (kpos >= lo || kpos < kept) && kpos <= pos;
        long long row = -1;
        float s = -INFINITY;
        if (valid) {
            int page = table[kpos / page_size];
            if (page < 0 || page >= total_pages) {
                ie_report(err, page < 0 ? IE_ERR_TABLE : IE_ERR_PAGE, page, token);
                valid = false;
            } else {
                row = ((long long)page * nkv + kvh) * page_size + (kpos % page_size);
                s = (hd % 8 == 0 ? dot_row(qs, k_cache + row * hd, hd) : dot_row_any(qs, k_cache + row * hd, hd)) * scale;
                if (softcap > 0.f) s = softcap * tanhf(s * inv_cap);
                if (log_r1 != nullptr) s -= log_r1[head] * log1pf(log_r2[head] * (float)(pos - kpos));
                if (bias_table != nullptr) s += bias_table[(size_t)head * bias_len + min(pos - kpos, bias_len - 1)];
            }
        }
        float m_new = m, p;
        if (gated) {
            p = valid ? 1.0f / (1.0f + expf(-(s + hb))) : 0.f;
        } else {
            m_new = fmaxf(m, warp_max(s));
            p = valid ? expf(s - m_new) : 0.f;
            float alpha = (m == -INFINITY) ? 0.f : expf(m - m_new);
            l = l * alpha + warp_sum(p);
#pragma unroll
            for (int i = 0; i < MAX_ACC; ++i) acc[i] *= alpha;
        }
        int count = min(32, pos - t0 + 1);
        for (int j = 0; j < count; ++j) {
            float pj = __shfl_sync(0xffffffffu, p, j);
            long long rj = __shfl_sync(0xffffffffu, row, j);
            if (rj < 0) continue;  // uniform across the warp
            const T* vrow = v_cache + rj * v_stride;
#pragma unroll
            for (int i = 0; i < MAX_ACC; ++i) {
                int d = lane + 32 * i;
                if (i < nacc && d < hdv) acc[i] = fmaf(pj, ie_load(vrow + d), acc[i]);
            }
        }
        m = m_new;
    }
    T* orow = out + (size_t)token * out_ld + (size_t)head * hdv;
    float inv = gated ? 1.0f : (l > 0.f ? 1.0f / l : 0.f);
    if (out_gate != nullptr && !gate_elements) inv *= 1.0f / (1.0f + expf(-out_gate[(size_t)token * gate_ld + head]));
#pragma unroll
    for (int i = 0; i < MAX_ACC; ++i) {
        int d = lane + 32 * i;
        if (i < nacc && d < hdv) {
            float f = inv;
            if (out_gate != nullptr && gate_elements)
                f *= 1.0f / (1.0f + expf(-out_gate[(size_t)token * gate_ld + (size_t)head * hdv + d]));
            ie_store(orow + d, acc[i] * f);
        }
    }
}
}  // namespace

IE_API int ie_paged_attention_generic(const void* q, const void* k_cache, const void* v_cache,
                                      int dtype, const int* block_tables, int table_width,
                                      const int* seq_of_token, const int* positions, void* out,
                                      int num_tokens, int nh, int nkv, int hd, int hdv, int v_stride,
                                      int page_size, int total_pages, float scale, int window, int chunk,
                                      const float* head_bias, const float* sinks, const float* out_gate,
                                      int gate_ld, float softcap, int keep_first, int gate_elements,
                                      const float* log_r1, const float* log_r2, const float* bias_table,
                                      int bias_len, int out_ld, int* err, void* stream) {
    if (num_tokens <= 0) return 0;
    if (hd < 1 || hdv < 1 || hdv > 32 * MAX_ACC || nkv <= 0 || nh % nkv != 0 || out_ld < nh * hdv) return (int)cudaErrorInvalidValue;
    if (keep_first < 0 || softcap < 0.f || (keep_first > 0 && chunk > 0)) return (int)cudaErrorInvalidValue;
    if ((log_r1 == nullptr) != (log_r2 == nullptr) || (bias_table != nullptr && bias_len < 1))
        return (int)cudaErrorInvalidValue;
    dim3 grid((nh + WARPS - 1) / WARPS, num_tokens);
    size_t smem = (size_t)WARPS * hd * sizeof(float);
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == IE_BF16)
        paged_attention_generic_kernel<<<grid, WARPS * 32, smem, s>>>(
            (const __nv_bfloat16*)q, (const __nv_bfloat16*)k_cache, (const __nv_bfloat16*)v_cache,
            block_tables, table_width, seq_of_token, positions, (__nv_bfloat16*)out,
            nh, nkv, hd, hdv, v_stride, page_size, total_pages, scale, window, chunk, head_bias, sinks, out_gate, gate_ld, softcap, keep_first,
            gate_elements, log_r1, log_r2, bias_table, bias_len, out_ld, err);
    else
        paged_attention_generic_kernel<<<grid, WARPS * 32, smem, s>>>(
            (const float*)q, (const float*)k_cache, (const float*)v_cache,
            block_tables, table_width, seq_of_token, positions, (float*)out,
            nh, nkv, hd, hdv, v_stride, page_size, total_pages, scale, window, chunk, head_bias, sinks, out_gate, gate_ld, softcap, keep_first,
            gate_elements, log_r1, log_r2, bias_table, bias_len, out_ld, err);
    return IE_LAUNCH_CHECK();
}
