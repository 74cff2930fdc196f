// Retention on a 32-bit projection [N, ld] = (heads * dim queries, heads * dim keys, heads * vdim values,
// heads * vdim gates): linear attention whose state decays by one constant per head,
//     S_t = decay S_(t-1) + k_t v_t^T,   o_t = q_scale S_t^T q_t,
// with queries and keys rotated by position (the first rot_dims entries of a head, by pairs (i, i +
// rot_dims / 2), from the 32-bit table of angles), every head's o divided by its root mean square over vdim
// (eps inside the root, no weight) and multiplied by silu(gate).  The state of a head is kept column by
// column ([vdim][dim], 32-bit) in the request's slot.  Built per (RT_D, RT_DV): dim and vdim rounded up to
// multiples of 16; up to 128 each.
//
//  * retention_step: requests that bring a few tokens each.  A block owns a head of a request: it holds
//    the state in registers (eight lanes a column), takes the tokens in order, and writes the normalised,
//    gated result.  Rotation, recurrence and read-out are this one kernel, all 32-bit.  The state is asked
//    for before the programmatic-launch wait: in one step nothing but this kernel writes it.
//  * retention_chunk_state, retention_scan, retention_chunk_out: prompt portions.  A request's tokens are
//    cut into chunks of 64, counted from the portion's first token.  With pw[n] = decay^n (a table worked
//    out in 64-bit): (1) each chunk by itself sums U = sum_j pw[n - 1 - j] k_j v_j^T; (2) S runs through
//    the chunks, S <- pw[n] S + U, leaving the state before each chunk in U's place; (3) a chunk's output
//    is pw[i + 1] S^T q_i + sum_(j <= i) pw[i - j] (q_i . k_j) v_j, normalised and gated where it is
//    written.  The products of (1) and (3) run on the tensor cores (mma.sync.m16n8k16, 32-bit sums) with
//    every operand, the state included, as two bfloat16 terms (its rounded value and the remainder:
//    hi hi + hi lo + lo hi), which keeps 16 bits of mantissa of each; (2) and all decays are 32-bit.
#include "common.cuh"
#include <math.h>

#ifndef RT_D
#define RT_D 64
#endif
#ifndef RT_DV
#define RT_DV 64
#endif

namespace {
constexpr int D = RT_D, DV = RT_DV;
static_assert(D % 16 == 0 && DV % 16 == 0 && D <= 128 && DV <= 128, "sizes");
constexpr int CHUNK = 64;

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ void mma_bf16(float* c, const unsigned* a, unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm_x4(unsigned* r, const void* p) {
    unsigned a = (unsigned)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldsm_x4_trans(unsigned* r, const void* p) {
    unsigned a = (unsigned)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ unsigned pack_bf16(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<unsigned*>(&v);
}
__device__ __forceinline__ float bf16_round(float x) { return __bfloat162float(__float2bfloat16_rn(x)); }
__device__ __forceinline__ float silu_f(float y) { return y / (1.0f + expf(-y)); }
__device__ __forceinline__ void split_store(bf16* hi, bf16* lo, float x) {
    bf16 h = __float2bfloat16_rn(x);
    *hi = h;
    *lo = __float2bfloat16_rn(x - __bfloat162float(h));
}

// Which request and which of its chunks the block's chunk number means; false: there are fewer chunks.
__device__ __forceinline__ bool find_chunk(const int* cu_q, int num_seqs, int number, int& seq, int& chunk) {
    for (seq = 0; seq < num_seqs; ++seq) {
        int n = (cu_q[seq + 1] - cu_q[seq] + CHUNK - 1) / CHUNK;
        if (number < n) { chunk = number; return true; }
        number -= n;
    }
    return false;
}

struct Heads {  // where a head's parts of a token's projection row are
    const float* proj;
    int ld, heads, dim, vdim, rot_dims;
    const float* table;
    int table_positions;
    __device__ const float* q(size_t n, int h) const { return proj + n * ld + (size_t)h * dim; }
    __device__ const float* k(size_t n, int h) const { return proj + n * ld + (size_t)(heads + h) * dim; }
    __device__ const float* v(size_t n, int h) const { return proj + n * ld + (size_t)2 * heads * dim + (size_t)h * vdim; }
    __device__ const float* g(size_t n, int h) const { return v(n, h) + (size_t)heads * vdim; }
    // entry d of a head's row x, rotated for position pos
    __device__ float rotated(const float* x, int d, int pos) const {
        int half = rot_dims >> 1;
        if (d >= rot_dims) return x[d];
        const float* cs = table + (size_t)pos * rot_dims;  // the angles' cosines, then their sines
        if (d < half) return x[d] * cs[d] - x[d + half] * cs[half + d];
        return x[d] * cs[d - half] + x[d - half] * cs[d];
    }
};

// ---- a few tokens per request ------------------------------------------------------------------

constexpr int STEP_THREADS = 256, STEP_MOST = 8;
constexpr int TPC = 8;                                  // lanes of a column
constexpr int NV = (D + 4 * TPC - 1) / (4 * TPC);       // pieces of four entries per lane and column
constexpr int COLS = STEP_THREADS / TPC;                // columns per round
constexpr int ROUNDS = (DV + COLS - 1) / COLS;

// grid: (heads, requests)
__global__ void __launch_bounds__(STEP_THREADS)
retention_step_kernel(Heads at, const int* __restrict__ ctx_lens, const float* __restrict__ powers,
                      float* __restrict__ state, long long state_stride, const int* __restrict__ slots,
                      const int* __restrict__ cu_q, float q_scale, float eps, bf16* __restrict__ out, int num_slots,
                      int* err) {
    __shared__ __align__(16) float qs[D], ks[D];
    __shared__ float vs[DV], os[DV], red[STEP_THREADS / 32];
    ie_pdl_trigger();
    int head = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x;
    int start = cu_q[seq], len = cu_q[seq + 1] - start, slot = slots[seq];
    const int dim = at.dim, vdim = at.vdim;
    bool ok = len > 0 && slot >= 0 && slot < num_slots;
    int pos0 = ctx_lens[seq] - len;
    if (ok && at.rot_dims > 0 && pos0 + len > at.table_positions) {
        if (tid == 0) ie_report(err, IE_ERR_POSITION, pos0 + len - 1, start);
        ok = false;
    }
    if (!ok) { ie_pdl_wait(); return; }
    float* S = state + (size_t)slot * state_stride + (size_t)head * vdim * dim;
    int sub = tid % TPC, col0 = tid / TPC;
    float s[ROUNDS][NV][4];
    const bool vec = dim % 4 == 0;
#pragma unroll
    for (int r = 0; r < ROUNDS; ++r) {
        int col = r * COLS + col0;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            int d = (i * TPC + sub) * 4;
            const float* p = S + (size_t)col * dim + d;
#pragma unroll
            for (int e = 0; e < 4; ++e) s[r][i][e] = 0.f;
            if (col >= vdim) continue;
            if (vec) {
                if (d < dim) {
                    float4 x = *reinterpret_cast<const float4*>(p);
                    s[r][i][0] = x.x; s[r][i][1] = x.y; s[r][i][2] = x.z; s[r][i][3] = x.w;
                }
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (d + e < dim) s[r][i][e] = p[e];
            }
        }
    }
    float decay = powers[(size_t)head * (CHUNK + 1) + 1];
    ie_pdl_wait();
    for (int t = 0; t < len; ++t) {
        size_t n = (size_t)(start + t);
        if (t > 0) __syncthreads();
        for (int i = tid; i < D; i += STEP_THREADS) {
            qs[i] = i < dim ? at.rotated(at.q(n, head), i, pos0 + t) : 0.f;
            ks[i] = i < dim ? at.rotated(at.k(n, head), i, pos0 + t) : 0.f;
        }
        for (int i = tid; i < DV; i += STEP_THREADS) vs[i] = i < vdim ? at.v(n, head)[i] : 0.f;
        float gate = tid < vdim ? at.g(n, head)[tid] : 0.f;
        __syncthreads();
        float rd[ROUNDS];
#pragma unroll
        for (int r = 0; r < ROUNDS; ++r) rd[r] = 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            int d = (i * TPC + sub) * 4;
            if (d >= D) break;
            float4 q4 = *reinterpret_cast<const float4*>(qs + d), k4 = *reinterpret_cast<const float4*>(ks + d);
#pragma unroll
            for (int r = 0; r < ROUNDS; ++r) {
                int col = r * COLS + col0;
                float u = col < DV ? vs[col] : 0.f;
                s[r][i][0] = fmaf(k4.x, u, s[r][i][0] * decay);
                s[r][i][1] = fmaf(k4.y, u, s[r][i][1] * decay);
                s[r][i][2] = fmaf(k4.z, u, s[r][i][2] * decay);
                s[r][i][3] = fmaf(k4.w, u, s[r][i][3] * decay);
                rd[r] = fmaf(s[r][i][0], q4.x, rd[r]);
                rd[r] = fmaf(s[r][i][1], q4.y, rd[r]);
                rd[r] = fmaf(s[r][i][2], q4.z, rd[r]);
                rd[r] = fmaf(s[r][i][3], q4.w, rd[r]);
            }
        }
#pragma unroll
        for (int o = TPC >> 1; o > 0; o >>= 1)
#pragma unroll
            for (int r = 0; r < ROUNDS; ++r) rd[r] += __shfl_xor_sync(0xffffffffu, rd[r], o);
        if (sub == 0)
#pragma unroll
            for (int r = 0; r < ROUNDS; ++r) {
                int col = r * COLS + col0;
                if (col < vdim) os[col] = rd[r] * q_scale;
            }
        __syncthreads();
        float y = tid < vdim ? os[tid] : 0.f;
        float ss = warp_sum(y * y);
        if ((tid & 31) == 0) red[tid >> 5] = ss;
        __syncthreads();
        if (tid < vdim) {
            float total = 0.f;
#pragma unroll
            for (int w = 0; w < (DV + 31) / 32; ++w) total += red[w];
            float inv = 1.0f / sqrtf(total / (float)vdim + eps);
            ie_store(out + (n * at.heads + head) * vdim + tid, y * inv * silu_f(gate));
        }
    }
#pragma unroll
    for (int r = 0; r < ROUNDS; ++r) {
        int col = r * COLS + col0;
        if (col >= vdim) continue;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            int d = (i * TPC + sub) * 4;
            float* p = S + (size_t)col * dim + d;
            if (vec) {
                if (d < dim) *reinterpret_cast<float4*>(p) = make_float4(s[r][i][0], s[r][i][1], s[r][i][2], s[r][i][3]);
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (d + e < dim) p[e] = s[r][i][e];
            }
        }
    }
}

// ---- prompt portions ---------------------------------------------------------------------------

constexpr int LDD = D + 8, LDV = DV + 8;  // rows 16 bytes longer: ldmatrix rows fall on different banks

__device__ __forceinline__ void split_store4(bf16* hi, bf16* lo, float4 x) {
    unsigned h0 = pack_bf16(x.x, x.y), h1 = pack_bf16(x.z, x.w);
    *reinterpret_cast<uint2*>(hi) = make_uint2(h0, h1);
    *reinterpret_cast<uint2*>(lo) = make_uint2(pack_bf16(x.x - bf16_round(x.x), x.y - bf16_round(x.y)),
                                               pack_bf16(x.z - bf16_round(x.z), x.w - bf16_round(x.w)));
}
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }

// A chunk's rows of queries or keys, rotated and times a factor per row, as two bfloat16 terms; rows
// beyond the chunk's tokens and entries beyond dim are zero.  `weight(j)` is the factor of row j.  Four
// entries at a time where sizes and addresses allow (`vec`), so that many loads are on their way together.
template <int THREADS, typename W>
__device__ __forceinline__ void bring_rotated(const Heads& at, bool vec, bool keys, int n0, int cnt, int pos0, int head,
                                              bf16* hi, bf16* lo, W weight) {
    const float* first = keys ? at.k((size_t)n0, head) : at.q((size_t)n0, head);
    if (vec) {
        constexpr int QUADS = D / 4;
        static_assert(CHUNK * QUADS % THREADS == 0, "whole rounds");
        const int half = at.rot_dims >> 1;
#pragma unroll 4
        for (int it = 0; it < CHUNK * QUADS / THREADS; ++it) {
            int i = it * THREADS + threadIdx.x, j = i / QUADS, d = (i - j * QUADS) * 4;
            float4 x = make_float4(0.f, 0.f, 0.f, 0.f), p = x, c = make_float4(1.f, 1.f, 1.f, 1.f), sn = x;
            float sign = 1.f;
            if (j < cnt && d < at.dim) {
                const float* row = first + (size_t)j * at.ld;
                x = load4(row + d);
                if (d < at.rot_dims) {
                    int a = d < half ? d : d - half;
                    const float* cs = at.table + (size_t)(pos0 + j) * at.rot_dims;
                    p = load4(row + (d < half ? d + half : a));
                    c = load4(cs + a);
                    sn = load4(cs + half + a);
                    sign = d < half ? -1.f : 1.f;
                }
            }
            float w = j < cnt ? weight(j) : 0.f;
            x.x = (x.x * c.x + sign * (p.x * sn.x)) * w;
            x.y = (x.y * c.y + sign * (p.y * sn.y)) * w;
            x.z = (x.z * c.z + sign * (p.z * sn.z)) * w;
            x.w = (x.w * c.w + sign * (p.w * sn.w)) * w;
            split_store4(hi + j * LDD + d, lo + j * LDD + d, x);
        }
        return;
    }
    for (int i = threadIdx.x; i < CHUNK * D; i += THREADS) {
        int j = i / D, d = i - j * D;
        float x = 0.f;
        if (j < cnt && d < at.dim) x = at.rotated(first + (size_t)j * at.ld, d, pos0 + j) * weight(j);
        split_store(hi + j * LDD + d, lo + j * LDD + d, x);
    }
}
template <int THREADS>
__device__ __forceinline__ void bring_values(const Heads& at, bool vec, int n0, int cnt, int head, bf16* hi, bf16* lo) {
    const float* first = at.v((size_t)n0, head);
    if (vec) {
        constexpr int QUADS = DV / 4;
        static_assert(CHUNK * QUADS % THREADS == 0, "whole rounds");
#pragma unroll 8
        for (int it = 0; it < CHUNK * QUADS / THREADS; ++it) {
            int i = it * THREADS + threadIdx.x, j = i / QUADS, d = (i - j * QUADS) * 4;
            float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
            if (j < cnt && d < at.vdim) x = load4(first + (size_t)j * at.ld + d);
            split_store4(hi + j * LDV + d, lo + j * LDV + d, x);
        }
        return;
    }
    for (int i = threadIdx.x; i < CHUNK * DV; i += THREADS) {
        int j = i / DV, d = i - j * DV;
        float x = (j < cnt && d < at.vdim) ? first[(size_t)j * at.ld + d] : 0.f;
        split_store(hi + j * LDV + d, lo + j * LDV + d, x);
    }
}

constexpr int STATE_THREADS = 256;
constexpr size_t STATE_SMEM = (size_t)2 * CHUNK * (LDD + LDV) * sizeof(bf16);

// grid: (chunks, heads).  u: [chunks, heads, vdim, dim].
__global__ void __launch_bounds__(STATE_THREADS)
retention_chunk_state_kernel(Heads at, const int* __restrict__ ctx_lens, const float* __restrict__ powers,
                             const int* __restrict__ cu_q, int num_seqs, bool vec, float* __restrict__ u,
                             int* err) {
    extern __shared__ __align__(16) unsigned char raw[];
    bf16* k_hi = reinterpret_cast<bf16*>(raw);
    bf16 *k_lo = k_hi + CHUNK * LDD, *v_hi = k_lo + CHUNK * LDD, *v_lo = v_hi + CHUNK * LDV;
    ie_pdl_trigger();
    ie_pdl_wait();
    int seq, chunk, head = blockIdx.y;
    if (!find_chunk(cu_q, num_seqs, blockIdx.x, seq, chunk)) return;
    int start = cu_q[seq], len = cu_q[seq + 1] - start, pos0 = ctx_lens[seq] - len + chunk * CHUNK;
    int n0 = start + chunk * CHUNK, cnt = min(CHUNK, len - chunk * CHUNK);
    if (at.rot_dims > 0 && pos0 + cnt > at.table_positions) {
        if (threadIdx.x == 0) ie_report(err, IE_ERR_POSITION, pos0 + cnt - 1, n0);
        return;
    }
    const float* pw = powers + (size_t)head * (CHUNK + 1);
    bring_rotated<STATE_THREADS>(at, vec, true, n0, cnt, pos0, head, k_hi, k_lo, [&](int j) { return pw[cnt - 1 - j]; });
    bring_values<STATE_THREADS>(at, vec, n0, cnt, head, v_hi, v_lo);
    __syncthreads();
    int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
    float* dst = u + ((size_t)blockIdx.x * at.heads + head) * at.vdim * at.dim;
    constexpr int WIDE = 32, NTASK = (D + WIDE - 1) / WIDE;
    for (int task = warp; task < (DV / 16) * NTASK; task += STATE_THREADS / 32) {
        int mt = task / NTASK, c0 = (task - mt * NTASK) * WIDE;
        float acc[WIDE / 8][4];
#pragma unroll
        for (int i = 0; i < WIDE / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
        for (int kk = 0; kk < CHUNK; kk += 16) {
            // A = V^T: 16 value entries x 16 tokens, from rows of tokens (transposed on the way)
            unsigned a_hi[4], a_lo[4];
            int arow = kk + (lane & 7) + ((lane >> 4) << 3), acol = mt * 16 + ((lane >> 3) & 1) * 8;
            ldsm_x4_trans(a_hi, v_hi + arow * LDV + acol);
            ldsm_x4_trans(a_lo, v_lo + arow * LDV + acol);
#pragma unroll
            for (int nt = 0; nt < WIDE / 8; nt += 2) {
                if (c0 + nt * 8 >= D) break;
                unsigned b_hi[4], b_lo[4];
                int brow = kk + (lane & 15), bcol = c0 + nt * 8 + (lane >> 4) * 8;
                ldsm_x4_trans(b_hi, k_hi + brow * LDD + bcol);
                ldsm_x4_trans(b_lo, k_lo + brow * LDD + bcol);
                mma_bf16(acc[nt], a_hi, b_hi[0], b_hi[1]);
                mma_bf16(acc[nt + 1], a_hi, b_hi[2], b_hi[3]);
                mma_bf16(acc[nt], a_lo, b_hi[0], b_hi[1]);
                mma_bf16(acc[nt + 1], a_lo, b_hi[2], b_hi[3]);
                mma_bf16(acc[nt], a_hi, b_lo[0], b_lo[1]);
                mma_bf16(acc[nt + 1], a_hi, b_lo[2], b_lo[3]);
            }
        }
        int r_a = mt * 16 + g, r_b = r_a + 8;
#pragma unroll
        for (int nt = 0; nt < WIDE / 8; ++nt) {
            int c2 = c0 + nt * 8 + t4 * 2;
            if (at.dim % 2 == 0) {
                if (c2 >= at.dim) continue;
                if (r_a < at.vdim) *reinterpret_cast<float2*>(dst + (size_t)r_a * at.dim + c2) = make_float2(acc[nt][0], acc[nt][1]);
                if (r_b < at.vdim) *reinterpret_cast<float2*>(dst + (size_t)r_b * at.dim + c2) = make_float2(acc[nt][2], acc[nt][3]);
                continue;
            }
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                int c = c2 + e;
                if (c < at.dim && r_a < at.vdim) dst[(size_t)r_a * at.dim + c] = acc[nt][e];
                if (c < at.dim && r_b < at.vdim) dst[(size_t)r_b * at.dim + c] = acc[nt][2 + e];
            }
        }
    }
}

// grid: (blocks of 256 * VEC entries, heads, requests): the state goes through a request's chunks.  The
// next few chunks' sums are on their way while the last ones are added.
template <int VEC>
__global__ void __launch_bounds__(256)
retention_scan_kernel(float* __restrict__ u, const float* __restrict__ powers, float* __restrict__ state,
                      long long state_stride, const int* __restrict__ slots, const int* __restrict__ cu_q, int heads,
                      int entries, int num_slots) {
    ie_pdl_trigger();
    ie_pdl_wait();
    int seq = blockIdx.z, head = blockIdx.y;
    int len = cu_q[seq + 1] - cu_q[seq], slot = slots[seq];
    if (len <= 0 || slot < 0 || slot >= num_slots) return;
    int first = 0;  // the request's first chunk among the step's
    for (int i = 0; i < seq; ++i) first += (cu_q[i + 1] - cu_q[i] + CHUNK - 1) / CHUNK;
    int e = (blockIdx.x * 256 + threadIdx.x) * VEC;
    if (e >= entries) return;
    int chunks = (len + CHUNK - 1) / CHUNK;
    const float* pw = powers + (size_t)head * (CHUNK + 1);
    float* S = state + (size_t)slot * state_stride + (size_t)head * entries + e;
    float* p = u + ((size_t)first * heads + head) * entries + e;
    const size_t step = (size_t)heads * entries;
    struct alignas(4 * VEC) Pack { float v[VEC]; };
    Pack s = *reinterpret_cast<const Pack*>(S);
    const float full = pw[CHUNK], last = pw[len - (chunks - 1) * CHUNK];
    constexpr int AHEAD = 8;
    Pack x[AHEAD];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i)
        if (i < chunks) x[i] = *reinterpret_cast<const Pack*>(p + (size_t)i * step);
    for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            int c = c0 + i;
            if (c >= chunks) break;
            Pack sum = x[i];
            if (c + AHEAD < chunks) x[i] = *reinterpret_cast<const Pack*>(p + (size_t)(c + AHEAD) * step);
            *reinterpret_cast<Pack*>(p + (size_t)c * step) = s;
            float d = c + 1 < chunks ? full : last;
#pragma unroll
            for (int v = 0; v < VEC; ++v) s.v[v] = fmaf(d, s.v[v], sum.v[v]);
        }
    }
    *reinterpret_cast<Pack*>(S) = s;
}

// eight warps: warp w takes the sixteen rows (w & 3) * 16 .. and one half of the value entries
constexpr int OUT_THREADS = 256;
constexpr int PAIRS = DV / 16, WARP_PAIRS = (PAIRS + 1) / 2, TILES = 2 * WARP_PAIRS;  // of sixteen value entries; of eight
constexpr int OUT_STATE = 2 * DV * LDD, OUT_KV = 2 * CHUNK * (LDD + LDV);  // bfloat16 numbers: used one after the other
constexpr size_t OUT_SMEM = (size_t)(2 * CHUNK * LDD + (OUT_STATE > OUT_KV ? OUT_STATE : OUT_KV)) * sizeof(bf16);

// grid: (chunks, heads).  s_before: the state before each chunk, [chunks, heads, vdim, dim].
__global__ void __launch_bounds__(OUT_THREADS)
retention_chunk_out_kernel(Heads at, const int* __restrict__ ctx_lens, const float* __restrict__ powers,
                           const float* __restrict__ s_before, const int* __restrict__ cu_q, int num_seqs,
                           bool vec, float q_scale, float eps, bf16* __restrict__ out) {
    extern __shared__ __align__(16) unsigned char raw[];
    __shared__ float pw[CHUNK + 1];
    __shared__ float squares[2][CHUNK];
    bf16* q_hi = reinterpret_cast<bf16*>(raw);
    bf16 *q_lo = q_hi + CHUNK * LDD, *rest = q_lo + CHUNK * LDD;
    ie_pdl_trigger();
    ie_pdl_wait();
    int seq, chunk, head = blockIdx.y;
    if (!find_chunk(cu_q, num_seqs, blockIdx.x, seq, chunk)) return;
    int start = cu_q[seq], len = cu_q[seq + 1] - start, pos0 = ctx_lens[seq] - len + chunk * CHUNK;
    int n0 = start + chunk * CHUNK, cnt = min(CHUNK, len - chunk * CHUNK);
    if (at.rot_dims > 0 && pos0 + cnt > at.table_positions) return;  // (reported by the kernel before)
    for (int i = threadIdx.x; i <= CHUNK; i += OUT_THREADS) pw[i] = powers[(size_t)head * (CHUNK + 1) + i];
    bring_rotated<OUT_THREADS>(at, vec, false, n0, cnt, pos0, head, q_hi, q_lo, [](int) { return 1.0f; });
    {
        bf16 *s_hi = rest, *s_lo = rest + DV * LDD;
        const float* src = s_before + ((size_t)blockIdx.x * at.heads + head) * at.vdim * at.dim;
        if (vec) {
            constexpr int QUADS = D / 4;
#pragma unroll 8
            for (int i = threadIdx.x; i < DV * QUADS; i += OUT_THREADS) {
                int c = i / QUADS, d = (i - c * QUADS) * 4;
                float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
                if (c < at.vdim && d < at.dim) x = load4(src + (size_t)c * at.dim + d);
                split_store4(s_hi + c * LDD + d, s_lo + c * LDD + d, x);
            }
        } else {
            for (int i = threadIdx.x; i < DV * D; i += OUT_THREADS) {
                int c = i / D, d = i - c * D;
                float x = (c < at.vdim && d < at.dim) ? src[(size_t)c * at.dim + d] : 0.f;
                split_store(s_hi + c * LDD + d, s_lo + c * LDD + d, x);
            }
        }
    }
    __syncthreads();
    int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
    const int wr = warp & 3, wc = warp >> 2, col0 = wc * WARP_PAIRS * 16;  // the warp's rows and first value entry
    const bool active = wr * 16 < cnt && col0 < DV;
    float o[TILES][4];
#pragma unroll
    for (int i = 0; i < TILES; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    const int arow = (wr * 16 + (lane & 15)) * LDD + (lane >> 4) * 8;  // a warp's 16 rows of queries
    const int brow = (lane & 7) + ((lane >> 4) << 3), bcol = ((lane >> 3) & 1) * 8;
    if (active) {  // what the state before the chunk holds: pw[i + 1] S^T q_i
        const bf16 *s_hi = rest, *s_lo = rest + DV * LDD;
#pragma unroll 2
        for (int kk = 0; kk < D; kk += 16) {
            unsigned a_hi[4], a_lo[4];
            ldsm_x4(a_hi, q_hi + arow + kk);
            ldsm_x4(a_lo, q_lo + arow + kk);
#pragma unroll
            for (int nt = 0; nt < TILES; nt += 2) {
                if (col0 + nt * 8 >= DV) break;
                unsigned b_hi[4], b_lo[4];
                ldsm_x4(b_hi, s_hi + (col0 + nt * 8 + brow) * LDD + kk + bcol);
                ldsm_x4(b_lo, s_lo + (col0 + nt * 8 + brow) * LDD + kk + bcol);
                mma_bf16(o[nt], a_hi, b_hi[0], b_hi[1]);
                mma_bf16(o[nt + 1], a_hi, b_hi[2], b_hi[3]);
                mma_bf16(o[nt], a_lo, b_hi[0], b_hi[1]);
                mma_bf16(o[nt + 1], a_lo, b_hi[2], b_hi[3]);
                mma_bf16(o[nt], a_hi, b_lo[0], b_lo[1]);
                mma_bf16(o[nt + 1], a_hi, b_lo[2], b_lo[3]);
            }
        }
    }
    const int r_a = wr * 16 + g, r_b = r_a + 8;
    {
        float f_a = pw[r_a + 1], f_b = pw[r_b + 1];
#pragma unroll
        for (int i = 0; i < TILES; ++i) { o[i][0] *= f_a; o[i][1] *= f_a; o[i][2] *= f_b; o[i][3] *= f_b; }
    }
    __syncthreads();  // everyone is done with the state: the chunk's keys and values take its place
    bf16 *k_hi = rest, *k_lo = k_hi + CHUNK * LDD, *v_hi = k_lo + CHUNK * LDD, *v_lo = v_hi + CHUNK * LDV;
    bring_rotated<OUT_THREADS>(at, vec, true, n0, cnt, pos0, head, k_hi, k_lo, [](int) { return 1.0f; });
    bring_values<OUT_THREADS>(at, vec, n0, cnt, head, v_hi, v_lo);
    __syncthreads();
    // sixteen keys at a time, up to the warp's last row
    for (int kt = 0; active && kt <= wr; ++kt) {
        float s[2][4];
#pragma unroll
        for (int i = 0; i < 2; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
#pragma unroll 4
        for (int kk = 0; kk < D; kk += 16) {
            unsigned a_hi[4], a_lo[4], b_hi[4], b_lo[4];
            ldsm_x4(a_hi, q_hi + arow + kk);
            ldsm_x4(a_lo, q_lo + arow + kk);
            ldsm_x4(b_hi, k_hi + (kt * 16 + brow) * LDD + kk + bcol);
            ldsm_x4(b_lo, k_lo + (kt * 16 + brow) * LDD + kk + bcol);
            mma_bf16(s[0], a_hi, b_hi[0], b_hi[1]);
            mma_bf16(s[1], a_hi, b_hi[2], b_hi[3]);
            mma_bf16(s[0], a_lo, b_hi[0], b_hi[1]);
            mma_bf16(s[1], a_lo, b_hi[2], b_hi[3]);
            mma_bf16(s[0], a_hi, b_lo[0], b_lo[1]);
            mma_bf16(s[1], a_hi, b_lo[2], b_lo[3]);
        }
        unsigned p_hi[4], p_lo[4];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            float w[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                int n = (e < 2 ? r_a : r_b) - (kt * 16 + i * 8 + t4 * 2 + (e & 1));
                w[e] = n >= 0 ? s[i][e] * pw[n] : 0.f;
            }
            p_hi[i * 2] = pack_bf16(w[0], w[1]);
            p_hi[i * 2 + 1] = pack_bf16(w[2], w[3]);
            p_lo[i * 2] = pack_bf16(w[0] - bf16_round(w[0]), w[1] - bf16_round(w[1]));
            p_lo[i * 2 + 1] = pack_bf16(w[2] - bf16_round(w[2]), w[3] - bf16_round(w[3]));
        }
#pragma unroll
        for (int nt = 0; nt < TILES; nt += 2) {
            if (col0 + nt * 8 >= DV) break;
            unsigned b_hi[4], b_lo[4];
            int at_v = (kt * 16 + (lane & 15)) * LDV + col0 + nt * 8 + (lane >> 4) * 8;
            ldsm_x4_trans(b_hi, v_hi + at_v);
            ldsm_x4_trans(b_lo, v_lo + at_v);
            mma_bf16(o[nt], p_hi, b_hi[0], b_hi[1]);
            mma_bf16(o[nt + 1], p_hi, b_hi[2], b_hi[3]);
            mma_bf16(o[nt], p_lo, b_hi[0], b_hi[1]);
            mma_bf16(o[nt + 1], p_lo, b_hi[2], b_hi[3]);
            mma_bf16(o[nt], p_hi, b_lo[0], b_lo[1]);
            mma_bf16(o[nt + 1], p_hi, b_lo[2], b_lo[3]);
        }
    }
    // unit root mean square over the value entries (the columns beyond vdim hold zeros), gate, write
    float ss_a = 0.f, ss_b = 0.f;
#pragma unroll
    for (int i = 0; i < TILES; ++i) {
#pragma unroll
        for (int e = 0; e < 4; ++e) o[i][e] *= q_scale;
        ss_a = fmaf(o[i][0], o[i][0], fmaf(o[i][1], o[i][1], ss_a));
        ss_b = fmaf(o[i][2], o[i][2], fmaf(o[i][3], o[i][3], ss_b));
    }
    ss_a += __shfl_xor_sync(0xffffffffu, ss_a, 1);
    ss_a += __shfl_xor_sync(0xffffffffu, ss_a, 2);
    ss_b += __shfl_xor_sync(0xffffffffu, ss_b, 1);
    ss_b += __shfl_xor_sync(0xffffffffu, ss_b, 2);
    if (t4 == 0) {
        squares[wc][r_a] = ss_a;
        squares[wc][r_b] = ss_b;
    }
    __syncthreads();  // the row's other half of the value entries is another warp's
    if (!active) return;
    ss_a = squares[0][r_a] + squares[1][r_a];
    ss_b = squares[0][r_b] + squares[1][r_b];
    float inv_a = 1.0f / sqrtf(ss_a / (float)at.vdim + eps), inv_b = 1.0f / sqrtf(ss_b / (float)at.vdim + eps);
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        int r = half ? r_b : r_a;
        if (r >= cnt) continue;
        size_t n = (size_t)(n0 + r);
        const float* gate = at.g(n, head);
        bf16* dst = out + (n * at.heads + head) * at.vdim;
        float inv = half ? inv_b : inv_a;
        if (vec) {  // (pairs: vdim and the gates' addresses are multiples of four)
#pragma unroll
            for (int i = 0; i < TILES; ++i) {
                int c = col0 + i * 8 + t4 * 2;
                if (c >= at.vdim) break;
                float2 g2 = *reinterpret_cast<const float2*>(gate + c);
                *reinterpret_cast<unsigned*>(dst + c) =
                    pack_bf16(o[i][half * 2] * inv * silu_f(g2.x), o[i][half * 2 + 1] * inv * silu_f(g2.y));
            }
            continue;
        }
#pragma unroll
        for (int i = 0; i < TILES; ++i)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                int c = col0 + i * 8 + t4 * 2 + e;
                if (c < at.vdim) ie_store(dst + c, o[i][half * 2 + e] * inv * silu_f(gate[c]));
            }
    }
}
}  // namespace

IE_API int ie_retention_dims(int* d, int* dv) {
    *d = D;
    *dv = DV;
    return CHUNK;
}

// powers: [heads, 65], decay^0 .. decay^64; out: bfloat16 [N, heads * vdim].  chunks == 0: requests of at
// most 8 tokens each (the step kernel); else at least as many chunks of 64 tokens as the step's requests
// have, and `scratch` holds [chunks, heads, vdim, dim] floats.
IE_API int ie_retention(const float* proj, int ld, int heads, int dim, int vdim, const float* table, int rot_dims,
                        int table_positions, const int* ctx_lens, const float* powers, float* state,
                        long long state_stride, const int* slots, const int* cu_q, int num_seqs, float q_scale,
                        float eps, void* out, int num_slots, int max_q_len, int chunks, float* scratch, int* err,
                        void* stream) {
    if (num_seqs <= 0) return 0;
    if (dim < 1 || vdim < 1 || dim > D || vdim > DV || heads < 1 || ld < 2 * heads * (dim + vdim) || rot_dims < 0 ||
        rot_dims % 2 || rot_dims > dim || (rot_dims > 0 && table == nullptr))
        return (int)cudaErrorInvalidValue;
    cudaStream_t s = (cudaStream_t)stream;
    Heads at{proj, ld, heads, dim, vdim, rot_dims, table, table_positions};
    if (chunks == 0) {
        if (max_q_len > STEP_MOST) return (int)cudaErrorInvalidValue;
        return ie_launch(retention_step_kernel, dim3(heads, num_seqs), dim3(STEP_THREADS), 0, s, at, ctx_lens,
                         powers, state, state_stride, slots, cu_q, q_scale, eps, (bf16*)out, num_slots, err);
    }
    if (scratch == nullptr) return (int)cudaErrorInvalidValue;
    static IePerDevice allowed_state, allowed_out;
    cudaError_t e = ie_allow_smem(allowed_state, retention_chunk_state_kernel, STATE_SMEM);
    if (e == cudaSuccess) e = ie_allow_smem(allowed_out, retention_chunk_out_kernel, OUT_SMEM);
    if (e != cudaSuccess) return (int)e;
    // 16-byte pieces everywhere: every head's rows, the halves of a rotation, the table and the scratch
    const bool vec = dim % 4 == 0 && vdim % 4 == 0 && rot_dims % 8 == 0 && ld % 4 == 0 &&
                     ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(table) |
                       reinterpret_cast<uintptr_t>(scratch)) % 16 == 0);
    int rc = ie_launch(retention_chunk_state_kernel, dim3(chunks, heads), dim3(STATE_THREADS), STATE_SMEM, s, at,
                       ctx_lens, powers, cu_q, num_seqs, vec, scratch, err);
    if (rc != 0) return rc;
    int entries = dim * vdim;
    if (vec && state_stride % 4 == 0 && reinterpret_cast<uintptr_t>(state) % 16 == 0)
        rc = ie_launch(retention_scan_kernel<4>, dim3((entries + 1023) / 1024, heads, num_seqs), dim3(256), 0, s, scratch,
                       powers, state, state_stride, slots, cu_q, heads, entries, num_slots);
    else
        rc = ie_launch(retention_scan_kernel<1>, dim3((entries + 255) / 256, heads, num_seqs), dim3(256), 0, s, scratch,
                       powers, state, state_stride, slots, cu_q, heads, entries, num_slots);
    if (rc != 0) return rc;
    return ie_launch(retention_chunk_out_kernel, dim3(chunks, heads), dim3(OUT_THREADS), OUT_SMEM, s, at, ctx_lens,
                     powers, (const float*)scratch, cu_q, num_seqs, vec, q_scale, eps, (bf16*)out);
}
