// Kernels of the latent attention mixer besides the attention itself (which is the general paged
// kernel with value rows inside the key rows, or the tensor-core kernel of latent_attention_mma.cu):
//
//  * latent_prep: from the 32-bit products of the mixer's input, per token, whichever of these are asked for:
//    the queries' unrotated parts and their rotated parts (turned, written behind the latent part of the
//    query rows the attention reads); the heads' output gates; the cached row: the latent (divided by
//    its root mean square, times a weight) followed by the shared rotated key part; the queries' own
//    latent (divided by its root mean square, times a weight), from which another product makes the queries.
//  * headwise_linear: out[n, h, :] = W[h] x[n, h, :] (times an optional factor per token and
//    head): the products that move the per-head key and value matrices to the query side.
//  * headwise_mma: the same on the tensor cores (bfloat16) for steps of up to some hundred tokens; it can
//    read the 32-bit queries themselves and turn their rotated parts on the way, so that a step that follows
//    the queries' product needs one launch for everything up to the attention.
//
// Rotation of the first rot_dims entries of the rotated part, a = position * frequency from the 32-bit table
// [positions, 2, rot_dims / 2] (cosines, then sines, with whatever factor the encoding has): entries 2i and
// 2i+1 form a pair, or (halves) entries i and i + rot_dims / 2; (u, v) -> (u cos a - v sin a, v cos a + u sin a);
// entries from rot_dims on pass unchanged.
// All arithmetic is 32-bit; results are rounded once to the output's dtype.
#include "common.cuh"

namespace {

// A row of a 32-bit product that may have come back in parts (of a split inner dimension): added in order.
struct Row {
    const float* p;
    int parts;
    size_t stride;
    __device__ __forceinline__ float operator[](int i) const {
        float v = p[i];
#pragma unroll 4
        for (int s = 1; s < parts; ++s) v += p[s * stride + i];
        return v;
    }
    __device__ __forceinline__ float4 four(int i) const {
        float4 v = *reinterpret_cast<const float4*>(p + i);
#pragma unroll 8
        for (int s = 1; s < parts; ++s) {
            float4 x = *reinterpret_cast<const float4*>(p + s * stride + i);
            v.x += x.x; v.y += x.y; v.z += x.z; v.w += x.w;
        }
        return v;
    }
    __device__ __forceinline__ Row at(int i) const { return Row{p + i, parts, stride}; }
};

// entry d of a rotated part `src`, turned by the angles at `cs` (null: not turned)
template <typename Src>
__device__ __forceinline__ float turned(const Src& src, int d, const float* cs, int rot_dims, int interleaved) {
    float v = src[d];
    if (cs == nullptr || d >= rot_dims) return v;
    int half = rot_dims / 2;
    int j = interleaved ? d >> 1 : (d < half ? d : d - half);
    bool second = interleaved ? (d & 1) != 0 : d >= half;
    float c = cs[j], s = cs[half + j];
    if (second) return fmaf(v, c, src[interleaved ? d - 1 : d - half] * s);
    return fmaf(v, c, -src[interleaved ? d + 1 : d + half] * s);
}

// What a call asks for is what has a pointer: queries (q), gates (gate_pre), the cached row (dkv and
// slot_mapping), the queries' latent (cq).  Each input is a row `*_ld` numbers long per token, in `parts` parts
// `part_stride` apart.
struct LatentIn {
    const float* q; int q_ld;
    const float* gate_pre; int gate_ld;
    const float* dkv; int dkv_ld;
    const float* cq; int cq_ld, q_rank;
    int parts; size_t part_stride;
    const float* norm_w;
    const float* cq_norm_w;
    float eps;
    bool fours;  // sizes and addresses of cq and dkv allow pieces of four
    __device__ Row row(const float* p, int ld, int n) const { return Row{p + (size_t)n * ld, parts, part_stride}; }
};

constexpr int LP_THREADS = 256;

template <typename T>
__global__ void __launch_bounds__(LP_THREADS)
latent_prep_kernel(LatentIn in, const int* __restrict__ positions,
                   const float* __restrict__ table, int rot_dims, int table_rows, int interleaved,
                   T* __restrict__ q_plain, T* __restrict__ q_abs, float* __restrict__ gate, T* __restrict__ cq_out,
                   T* __restrict__ cache, const int* __restrict__ slot_mapping, int heads, int dim, int rot_dim,
                   int rank, int total_slots, int* err) {
    extern __shared__ __align__(16) float rows[];  // the queries' latent, then the cached row, as they come
    __shared__ float red[2][LP_THREADS / 32];
    ie_pdl_trigger();
    ie_pdl_wait();
    int n = blockIdx.x, tid = threadIdx.x;
    int hq = dim + rot_dim, krow = rank + rot_dim;
    int pos = positions[n];
    bool turn = table != nullptr && rot_dims > 0;
    if (turn && (pos < 0 || pos >= table_rows)) {
        if (tid == 0) ie_report(err, IE_ERR_POSITION, pos, n);
        turn = false;
    }
    const float* cs = turn ? table + (size_t)pos * rot_dims : nullptr;  // cos [rot_dims/2], then sin

    if (in.q != nullptr) {
        // queries: unrotated parts as they are, rotated parts behind the latent part of the query rows
        const Row row = in.row(in.q, in.q_ld, n);
        for (int i = tid; i < heads * dim; i += LP_THREADS) {
            int h = i / dim, d = i - h * dim;
            ie_store(q_plain + (size_t)n * heads * dim + i, row[h * hq + d]);
        }
        for (int i = tid; i < heads * rot_dim; i += LP_THREADS) {
            int h = i / rot_dim, d = i - h * rot_dim;
            ie_store(q_abs + ((size_t)n * heads + h) * krow + rank + d, turned(row.at(h * hq + dim), d, cs, rot_dims, interleaved));
        }
    }
    if (in.gate_pre != nullptr) {
        const Row g = in.row(in.gate_pre, in.gate_ld, n);
        for (int h = tid; h < heads; h += LP_THREADS) gate[(size_t)n * heads + h] = 1.0f / (1.0f + expf(-g[h]));
    }
    int slot = in.dkv != nullptr && slot_mapping != nullptr ? slot_mapping[n] : -1;
    bool cached = in.dkv != nullptr && slot_mapping != nullptr;  // (a run that borrows another layer's cache writes none)
    if (cached && (slot < 0 || slot >= total_slots)) {
        if (tid == 0) ie_report(err, IE_ERR_PAGE, slot, n);
        cached = false;
    }
    const int n_cq = in.cq != nullptr ? in.q_rank : 0, n_row = cached ? krow : 0;
    if (n_cq + n_row == 0) return;
    const Row cq = in.row(in.cq, in.cq_ld, n), dkv = in.row(in.dkv, in.dkv_ld, n);
    float ss_q = 0.f, ss_c = 0.f;
    if (in.fours) {
#pragma unroll 2
        for (int i = tid * 4; i < n_cq + n_row; i += LP_THREADS * 4) {
            float4 v = i < n_cq ? cq.four(i) : dkv.four(i - n_cq);
            *reinterpret_cast<float4*>(rows + i) = v;
            float s = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w)));
            if (i < n_cq) ss_q += s;
            else if (i - n_cq < rank) ss_c += s;
        }
    } else {
        for (int i = tid; i < n_cq + n_row; i += LP_THREADS) {
            float v = i < n_cq ? cq[i] : dkv[i - n_cq];
            rows[i] = v;
            if (i < n_cq) ss_q = fmaf(v, v, ss_q);
            else if (i - n_cq < rank) ss_c = fmaf(v, v, ss_c);
        }
    }
    ss_q = warp_sum(ss_q);
    ss_c = warp_sum(ss_c);
    if ((tid & 31) == 0) { red[0][tid >> 5] = ss_q; red[1][tid >> 5] = ss_c; }
    __syncthreads();
    ss_q = ss_c = 0.f;
#pragma unroll
    for (int w = 0; w < LP_THREADS / 32; ++w) { ss_q += red[0][w]; ss_c += red[1][w]; }
    const float inv_q = n_cq > 0 ? 1.0f / sqrtf(ss_q / (float)n_cq + in.eps) : 0.f;
    const float inv_c = 1.0f / sqrtf(ss_c / (float)rank + in.eps);
    T* dst = cache + (size_t)max(slot, 0) * krow;
    const float* part = rows + n_cq + rank;
    for (int i = tid; i < n_cq + n_row; i += LP_THREADS) {
        if (i < n_cq) ie_store(cq_out + (size_t)n * n_cq + i, rows[i] * inv_q * in.cq_norm_w[i]);
        else if (i - n_cq < rank) ie_store(dst + i - n_cq, rows[i] * inv_c * in.norm_w[i - n_cq]);
        else ie_store(dst + i - n_cq, turned(part, i - n_cq - rank, cs, rot_dims, interleaved));
    }
}

// out[n, h, o] = scale[n, h] * sum_k x[n, h, k] * W[h, o, k], k ascending per output.
// x rows: x + n * x_ld + h * x_hs; out rows: out + n * o_ld + h * o_hs.  Tiles of 32 tokens x 32
// outputs of one head; each of 256 threads owns a 2 x 2 patch.
constexpr int HB = 32, HK = 32;

template <typename T>
__global__ void __launch_bounds__(256)
headwise_linear_kernel(const T* __restrict__ x, long long x_ld, long long x_hs, const T* __restrict__ w,
                       T* __restrict__ out, long long o_ld, long long o_hs,
                       const float* __restrict__ scale, int N, int heads, int O, int K) {
    __shared__ float xs[HK][HB + 1];
    __shared__ float ws[HK][HB + 1];
    ie_pdl_trigger();
    ie_pdl_wait();
    int h = blockIdx.z, n0 = blockIdx.y * HB, o0 = blockIdx.x * HB;
    int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const T* wh = w + (size_t)h * O * K;
    float acc[2][2] = {{0.f, 0.f}, {0.f, 0.f}};
    for (int k0 = 0; k0 < K; k0 += HK) {
        for (int i = tid; i < HB * HK; i += 256) {
            int r = i / HK, k = i - r * HK;
            float xv = 0.f, wv = 0.f;
            if (k0 + k < K) {
                if (n0 + r < N) xv = ie_load(x + (size_t)(n0 + r) * x_ld + (size_t)h * x_hs + k0 + k);
                if (o0 + r < O) wv = ie_load(wh + (size_t)(o0 + r) * K + k0 + k);
            }
            xs[k][r] = xv;
            ws[k][r] = wv;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < HK; ++k) {
            float a0 = xs[k][ty * 2], a1 = xs[k][ty * 2 + 1], b0 = ws[k][tx * 2], b1 = ws[k][tx * 2 + 1];
            acc[0][0] = fmaf(a0, b0, acc[0][0]); acc[0][1] = fmaf(a0, b1, acc[0][1]);
            acc[1][0] = fmaf(a1, b0, acc[1][0]); acc[1][1] = fmaf(a1, b1, acc[1][1]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        int n = n0 + ty * 2 + i;
        if (n >= N) continue;
        float f = scale ? scale[(size_t)n * heads + h] : 1.0f;
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            int o = o0 + tx * 2 + j;
            if (o < O) ie_store(out + (size_t)n * o_ld + (size_t)h * o_hs + o, acc[i][j] * f);
        }
    }
}
// out[n, h, :] *= scale[n, h] (bfloat16 rows of `o` entries, rows n * o_ld + h * o_hs apart)
__global__ void scale_head_rows_kernel(__nv_bfloat16* __restrict__ out, long long o_ld, long long o_hs,
                                       const float* __restrict__ scale, int heads, int o) {
    ie_pdl_trigger();
    ie_pdl_wait();
    int n = blockIdx.x;
    for (int i = threadIdx.x; i < heads * o; i += blockDim.x) {
        int h = i / o, c = i - h * o;
        __nv_bfloat16* p = out + (size_t)n * o_ld + (size_t)h * o_hs + c;
        *p = __float2bfloat16_rn(__bfloat162float(*p) * scale[(size_t)n * heads + h]);
    }
}

// The same products on the tensor cores (bfloat16 weights, K a multiple of 16): W's rows are the
// instruction's 16 rows, tokens its columns.  XT float: x is the queries' 32-bit product (rounded to bfloat16
// here; in `x_parts` parts x_stride apart), and a head's last block turns the rotated part that follows x in its row
// (`rot`).  A block of four warps takes either 64 outputs, a warp each sixteen (SPLIT false), or sixteen
// outputs with K cut among its warps, whose sums are added in order (SPLIT true: long K, few outputs).
// grid: (output blocks, heads, blocks of 8 * NT tokens).
struct RotatedPart {
    const int* positions;
    const float* table;
    int rot_dims, table_rows, interleaved, rot_dim, at;  // the part starts `at` entries behind x; 0 entries: none
    int dst_at;                                           // ... and goes so many entries behind out
    int* err;
};

__device__ __forceinline__ void mma_m16n8k16(float* c, const unsigned* a, unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

template <typename XT, int NT, bool SPLIT>
__global__ void __launch_bounds__(128)
headwise_mma_kernel(const XT* __restrict__ x, long long x_ld, long long x_hs, const __nv_bfloat16* __restrict__ w,
                    __nv_bfloat16* __restrict__ out, long long o_ld, long long o_hs, const float* __restrict__ scale,
                    RotatedPart rot, int x_parts, long long x_stride, bool fours, int N, int heads, int O, int K) {
    extern __shared__ __align__(16) unsigned char raw[];
    __nv_bfloat16* xs = reinterpret_cast<__nv_bfloat16*>(raw);  // [8 * NT][K + 8]
    float* sums = reinterpret_cast<float*>(xs + 8 * NT * (K + 8));  // SPLIT: [4][16][8 * NT]
    ie_pdl_trigger();
    const int h = blockIdx.y, n0 = blockIdx.z * 8 * NT, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int g = lane >> 2, t4 = lane & 3, ld = K + 8;
    const int o0 = SPLIT ? blockIdx.x * 16 : (blockIdx.x * 4 + warp) * 16;
    const int steps = K / 16, k_begin = SPLIT ? warp * steps / 4 : 0, k_end = SPLIT ? (warp + 1) * steps / 4 : steps;
    // A thread's four consecutive entries of a row are the instruction's columns 2 t4, 2 t4 + 1 and 2 t4 + 8, 2 t4 + 9:
    // the same renaming of k for both operands.  The first steps' weights, which no kernel writes, are asked for
    // before the wait.
    const __nv_bfloat16* wa = w + ((size_t)h * O + (o0 + g < O ? o0 + g : 0)) * K + t4 * 4;
    const __nv_bfloat16* wb = w + ((size_t)h * O + (o0 + g + 8 < O ? o0 + g + 8 : 0)) * K + t4 * 4;
    constexpr int EARLY = 8;
    uint2 ra[EARLY], rb[EARLY];
#pragma unroll
    for (int i = 0; i < EARLY; ++i)
        if (k_begin + i < k_end) {
            ra[i] = *reinterpret_cast<const uint2*>(wa + (k_begin + i) * 16);
            rb[i] = *reinterpret_cast<const uint2*>(wb + (k_begin + i) * 16);
        }
    ie_pdl_wait();
    const int cnt = min(8 * NT, N - n0);
    if (rot.rot_dim > 0 && blockIdx.x + 1 == gridDim.x) {
        for (int i = tid; i < cnt * rot.rot_dim; i += 128) {
            int r = i / rot.rot_dim, d = i - r * rot.rot_dim, pos = rot.positions[n0 + r];
            bool turn = rot.table != nullptr && rot.rot_dims > 0;
            if (turn && (pos < 0 || pos >= rot.table_rows)) {
                if (d == 0) ie_report(rot.err, IE_ERR_POSITION, pos, n0 + r);
                turn = false;
            }
            const XT* p = x + (size_t)(n0 + r) * x_ld + (size_t)h * x_hs + rot.at;
            float v = 0.f;
            if constexpr (sizeof(XT) == 4)
                v = turned(Row{p, x_parts, (size_t)x_stride}, d, turn ? rot.table + (size_t)pos * rot.rot_dims : nullptr, rot.rot_dims, rot.interleaved);
            out[(size_t)(n0 + r) * o_ld + (size_t)h * o_hs + rot.dst_at + d] = __float2bfloat16_rn(v);
        }
        return;
    }
    for (int i = tid; i < 8 * NT * (K / 4); i += 128) {
        int r = i / (K / 4), c = (i - r * (K / 4)) * 4;
        uint2 v = make_uint2(0u, 0u);
        if (r < cnt) {
            const XT* p = x + (size_t)(n0 + r) * x_ld + (size_t)h * x_hs + c;
            if constexpr (sizeof(XT) == 4) {
                float4 f;
                if (fours) {
                    f = Row{p, x_parts, (size_t)x_stride}.four(0);
                } else {
                    const Row all{p, x_parts, (size_t)x_stride};
                    f = make_float4(all[0], all[1], all[2], all[3]);
                }
                __nv_bfloat162 lo = __floats2bfloat162_rn(f.x, f.y), hi = __floats2bfloat162_rn(f.z, f.w);
                v = make_uint2(*reinterpret_cast<unsigned*>(&lo), *reinterpret_cast<unsigned*>(&hi));
            } else if (fours) {
                v = *reinterpret_cast<const uint2*>(p);
            } else {
                __nv_bfloat162 lo = __halves2bfloat162(p[0], p[1]), hi = __halves2bfloat162(p[2], p[3]);
                v = make_uint2(*reinterpret_cast<unsigned*>(&lo), *reinterpret_cast<unsigned*>(&hi));
            }
        }
        *reinterpret_cast<uint2*>(xs + r * ld + c) = v;
    }
    __syncthreads();
    float c[NT][4];
#pragma unroll
    for (int t = 0; t < NT; ++t) c[t][0] = c[t][1] = c[t][2] = c[t][3] = 0.f;
    if (o0 < O) {
        auto step = [&](int kk, uint2 pa, uint2 pb) {
            unsigned a[4] = {pa.x, pb.x, pa.y, pb.y};
#pragma unroll
            for (int t = 0; t < NT; ++t) {
                uint2 b = *reinterpret_cast<const uint2*>(xs + (t * 8 + g) * ld + kk * 16 + t4 * 4);
                mma_m16n8k16(c[t], a, b.x, b.y);
            }
        };
#pragma unroll
        for (int i = 0; i < EARLY; ++i)
            if (k_begin + i < k_end) step(k_begin + i, ra[i], rb[i]);
#pragma unroll 8
        for (int kk = k_begin + EARLY; kk < k_end; ++kk)
            step(kk, *reinterpret_cast<const uint2*>(wa + kk * 16), *reinterpret_cast<const uint2*>(wb + kk * 16));
    }
    if constexpr (SPLIT) {
#pragma unroll
        for (int t = 0; t < NT; ++t) {
            float* dst = sums + (warp * 16 + g) * 8 * NT + t * 8 + t4 * 2;
            dst[0] = c[t][0]; dst[1] = c[t][1];
            dst[64 * NT] = c[t][2]; dst[64 * NT + 1] = c[t][3];
        }
        __syncthreads();
        for (int i = tid; i < 16 * 8 * NT; i += 128) {
            int o = i % 16, r = i / 16, at = o * 8 * NT + r;
            if (r >= cnt || o0 + o >= O) continue;
            float v = ((sums[at] + sums[128 * NT + at]) + sums[256 * NT + at]) + sums[384 * NT + at];
            if (scale) v *= scale[(size_t)(n0 + r) * heads + h];
            out[(size_t)(n0 + r) * o_ld + (size_t)h * o_hs + o0 + o] = __float2bfloat16_rn(v);
        }
    } else {
#pragma unroll
        for (int t = 0; t < NT; ++t)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                int o = o0 + g + (e >> 1) * 8, r = t * 8 + t4 * 2 + (e & 1);
                if (o >= O || r >= cnt) continue;
                float v = c[t][e];
                if (scale) v *= scale[(size_t)(n0 + r) * heads + h];
                out[(size_t)(n0 + r) * o_ld + (size_t)h * o_hs + o] = __float2bfloat16_rn(v);
            }
    }
}

template <typename XT, int NT, bool SPLIT>
int launch_headwise_mma(const void* x, long long x_ld, long long x_hs, const void* w, void* out, long long o_ld,
                        long long o_hs, const float* scale, RotatedPart rot, int x_parts, long long x_stride, int N,
                        int heads, int O, int K, cudaStream_t s) {
    size_t smem = (size_t)8 * NT * (K + 8) * 2 + (SPLIT ? (size_t)4 * 16 * 8 * NT * 4 : 0);
    static IePerDevice allowed;
    cudaError_t e = ie_allow_smem(allowed, headwise_mma_kernel<XT, NT, SPLIT>, 96 * 1024);
    if (e != cudaSuccess) return (int)e;
    const bool fours = x_ld % 4 == 0 && x_hs % 4 == 0 && x_stride % 4 == 0 && reinterpret_cast<uintptr_t>(x) % (4 * sizeof(XT)) == 0;
    dim3 grid((SPLIT ? (O + 15) / 16 : (O + 63) / 64) + (rot.rot_dim > 0 ? 1 : 0), heads, (N + 8 * NT - 1) / (8 * NT));
    return ie_launch(headwise_mma_kernel<XT, NT, SPLIT>, grid, dim3(128), smem, s, (const XT*)x, x_ld, x_hs,
                     (const __nv_bfloat16*)w, (__nv_bfloat16*)out, o_ld, o_hs, scale, rot, x_parts, x_stride, fours, N, heads, O, K);
}

template <typename XT>
int pick_headwise_mma(const void* x, long long x_ld, long long x_hs, const void* w, void* out, long long o_ld,
                      long long o_hs, const float* scale, RotatedPart rot, int x_parts, long long x_stride, int N,
                        int heads, int O, int K, cudaStream_t s) {
#define IE_HM_ARGS x, x_ld, x_hs, w, out, o_ld, o_hs, scale, rot, x_parts, x_stride, N, heads, O, K, s
    // (the cut must not change with the number of tokens: a token's sums depend on the sizes alone)
    bool split = K >= 256;
    if (N <= 8) return split ? launch_headwise_mma<XT, 1, true>(IE_HM_ARGS) : launch_headwise_mma<XT, 1, false>(IE_HM_ARGS);
    return split ? launch_headwise_mma<XT, 4, true>(IE_HM_ARGS) : launch_headwise_mma<XT, 4, false>(IE_HM_ARGS);
#undef IE_HM_ARGS
}
}  // namespace

IE_API int ie_scale_head_rows(void* out, long long o_ld, long long o_hs, const float* scale, int N, int heads, int o,
                              void* stream) {
    if (N <= 0) return 0;
    return ie_launch(scale_head_rows_kernel, dim3(N), dim3(256), 0, (cudaStream_t)stream, (__nv_bfloat16*)out, o_ld, o_hs,
                     scale, heads, o);
}

IE_API int ie_latent_prep(const float* q, int q_ld, const float* gate_pre, int gate_ld, const float* dkv, int dkv_ld,
                          const float* cq, int cq_ld, int q_rank, int parts, long long part_stride, const float* norm_w, const float* cq_norm_w, float eps,
                          const int* positions, const float* table, int rot_dims, int table_rows, int interleaved,
                          void* q_plain, void* q_abs, float* gate, void* cq_out, void* cache, int dtype,
                          const int* slot_mapping, int num_tokens, int heads, int dim, int rot_dim, int rank,
                          int total_slots, int* err, void* stream) {
    if (num_tokens <= 0) return 0;
    if (rot_dims < 0 || rot_dims % 2 || rot_dims > rot_dim) return (int)cudaErrorInvalidValue;
    cudaStream_t s = (cudaStream_t)stream;
    if (parts < 1) return (int)cudaErrorInvalidValue;
    LatentIn in{q, q_ld, gate_pre, gate_ld, dkv, dkv_ld, cq, cq_ld, q_rank, parts, (size_t)part_stride, norm_w, cq_norm_w, eps, false};
    in.fours = q_rank % 4 == 0 && rank % 4 == 0 && rot_dim % 4 == 0 && cq_ld % 4 == 0 && dkv_ld % 4 == 0 && part_stride % 4 == 0 &&
               ((reinterpret_cast<uintptr_t>(cq) | reinterpret_cast<uintptr_t>(dkv)) % 16 == 0);
    size_t smem = ((cq ? q_rank : 0) + (dkv ? rank + rot_dim : 0)) * sizeof(float);
    if (smem > 40 * 1024) return (int)cudaErrorInvalidValue;
    if (dtype == IE_BF16)
        return ie_launch(latent_prep_kernel<__nv_bfloat16>, dim3(num_tokens), dim3(LP_THREADS), smem, s, in, positions, table,
                         rot_dims, table_rows, interleaved, (__nv_bfloat16*)q_plain, (__nv_bfloat16*)q_abs, gate,
                         (__nv_bfloat16*)cq_out, (__nv_bfloat16*)cache, slot_mapping, heads, dim, rot_dim, rank,
                         total_slots, err);
    return ie_launch(latent_prep_kernel<float>, dim3(num_tokens), dim3(LP_THREADS), smem, s, in, positions, table, rot_dims,
                     table_rows, interleaved, (float*)q_plain, (float*)q_abs, gate, (float*)cq_out, (float*)cache,
                     slot_mapping, heads, dim, rot_dim, rank, total_slots, err);
}

// Whether headwise_mma takes this inner size (else headwise_linear runs).
IE_API int ie_headwise_mma_ok(int K) { return K % 16 == 0 && K >= 16 && K <= 1024; }

// x: bfloat16, or 32-bit (x_f32) with a rotated part of rot_dim entries that starts `rot_at` entries behind x.
IE_API int ie_headwise_mma(const void* x, int x_f32, long long x_ld, long long x_hs, const void* w, void* out,
                           long long o_ld, long long o_hs, const float* scale, int N, int heads, int O, int K,
                           int x_parts, long long x_stride, const int* positions, const float* table, int rot_dims,
                           int table_rows, int interleaved, int rot_dim, int rot_at, int rot_dst, int* err, void* stream) {
    if (N <= 0 || heads <= 0 || O <= 0) return 0;
    if (!ie_headwise_mma_ok(K) || x_parts < 1 || (rot_dim > 0 && (!x_f32 || positions == nullptr)) || rot_dims < 0 || rot_dims % 2 ||
        rot_dims > rot_dim || reinterpret_cast<uintptr_t>(w) % 8)
        return (int)cudaErrorInvalidValue;
    RotatedPart rot{positions, table, rot_dims, table_rows, interleaved, rot_dim, rot_at, rot_dst, err};
    cudaStream_t s = (cudaStream_t)stream;
    if (x_f32) return pick_headwise_mma<float>(x, x_ld, x_hs, w, out, o_ld, o_hs, scale, rot, x_parts, x_stride, N, heads, O, K, s);
    return pick_headwise_mma<__nv_bfloat16>(x, x_ld, x_hs, w, out, o_ld, o_hs, scale, rot, x_parts, x_stride, N, heads, O, K, s);
}

IE_API int ie_headwise_linear(const void* x, long long x_ld, long long x_hs, const void* w, void* out,
                              long long o_ld, long long o_hs, const float* scale, int dtype, int N, int heads,
                              int O, int K, void* stream) {
    if (N <= 0 || heads <= 0 || O <= 0) return 0;
    dim3 grid((O + HB - 1) / HB, (N + HB - 1) / HB, heads);
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == IE_BF16)
        return ie_launch(headwise_linear_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, (const __nv_bfloat16*)x, x_ld,
                         x_hs, (const __nv_bfloat16*)w, (__nv_bfloat16*)out, o_ld, o_hs, scale, N, heads, O, K);
    return ie_launch(headwise_linear_kernel<float>, grid, dim3(256), 0, s, (const float*)x, x_ld, x_hs,
                     (const float*)w, (float*)out, o_ld, o_hs, scale, N, heads, O, K);
}
