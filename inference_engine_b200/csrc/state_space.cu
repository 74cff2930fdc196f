// State-space duality (Mamba-2) in the bfloat16 path: per head of a request
//     S_t = a_t S_(t-1) + dt_t B_t x_t^T,   y_t = S_t^T C_t + D x_t,   times silu(z_t),
// with S of N x P kept column by column ([P][N], 32-bit) in the request's slot, a_t = exp(-exp(A_log) dt_t), dt_t =
// softplus(. + dt_bias), and B, C shared by the heads of a group.  x, B and C are a short convolution of the
// projection with bias and silu, rounded to bfloat16 (in both forms below alike); a projection row is (z: heads *
// P, x: heads * P, B: groups * N, C: groups * N, dt: heads), 32-bit.  y goes out in 32-bit: the norm over parts of
// the row that follows needs all heads.  Built per (SS_N, SS_P): N and P rounded up to multiples of 16; up to 128
// each.
//
//  * state_space_step: requests that bring a few tokens each.  A block owns a head of a request: it holds the state
//    in registers (eight lanes a column), takes the tokens in order, and does convolution, step sizes,
//    recurrence, skip and gate itself.  (The slot's kept convolution inputs are read here and moved on by the norm's
//    kernel: the blocks of a group's heads all read the group's.)
//  * chunk_state, chunk_scan, chunk_out: prompt portions, after the convolution has been written out.  A request's
//    tokens are cut into chunks of 64, counted from the portion's first token.  With l_i the sum of log a over the
//    chunk up to token i: (1) each chunk by itself sums U = sum_j exp(l_last - l_j) dt_j B_j x_j^T; (2) S runs
//    through the chunks, S <- exp(l_last) S + U, leaving the state before each chunk as two bfloat16 terms (its
//    rounded value and the remainder); (3) a chunk's output is exp(l_i) S^T C_i + sum_(j <= i) exp(l_i - l_j) dt_j
//    (C_i . B_j) x_j.  The products of (1) and (3) run on the tensor cores (mma.sync.m16n8k16, 32-bit sums): B, C and
//    x are bfloat16 as they are, whatever else enters (the state, x times its step and decay, weighted scores) goes
//    in as two bfloat16 terms, which keeps 16 bits of mantissa; decays, step sizes and (2) are 32-bit.
#include "common.cuh"
#include <math.h>

#ifndef SS_N
#define SS_N 64
#endif
#ifndef SS_P
#define SS_P 64
#endif

namespace {
constexpr int D = SS_N, DV = SS_P;
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
__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool there) {
    unsigned d = (unsigned)__cvta_generic_to_shared(dst);
    int bytes = there ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_async_all() {
    asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group 0;" ::: "memory");
}
__device__ __forceinline__ unsigned pack_bf16(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<unsigned*>(&v);
}
__device__ __forceinline__ float bf16_round(float x) { return __bfloat162float(__float2bfloat16_rn(x)); }
__device__ __forceinline__ float silu_f(float y) { return y / (1.0f + expf(-y)); }
__device__ __forceinline__ float softplus_f(float y) { return y > 20.0f ? y : log1pf(expf(y)); }

struct Sizes {
    int heads, groups, n, p;  // n: state rows, p: value entries of a head
    __device__ int inner() const { return heads * p; }
    __device__ int channels() const { return heads * p + 2 * groups * n; }
    // columns of the convolved row
    __device__ int x_at(int head) const { return head * p; }
    __device__ int b_at(int head) const { return heads * p + head / (heads / groups) * n; }
    __device__ int c_at(int head) const { return heads * p + (groups + head / (heads / groups)) * n; }
};

// Which request and which of its chunks the block's chunk number means; false: there are fewer chunks.
__device__ __forceinline__ bool find_chunk(const int* cu_q, int num_seqs, int number, int& seq, int& chunk) {
    for (seq = 0; seq < num_seqs; ++seq) {
        int n = (cu_q[seq + 1] - cu_q[seq] + CHUNK - 1) / CHUNK;
        if (number < n) { chunk = number; return true; }
        number -= n;
    }
    return false;
}

// ---- a few tokens per request ------------------------------------------------------------------

constexpr int STEP_THREADS = 256, STEP_MOST = 8;
constexpr int TPC = 8;                                  // lanes of a column
constexpr int NV = (D + 4 * TPC - 1) / (4 * TPC);       // pieces of four entries per lane and column
constexpr int COLS = STEP_THREADS / TPC;                // columns per round
constexpr int ROUNDS = (DV + COLS - 1) / COLS;

// grid: (heads, requests).  proj: the projection's rows, `ld` numbers apart; y: [N, heads * p].
__global__ void __launch_bounds__(STEP_THREADS)
state_space_step_kernel(Sizes at, const float* __restrict__ proj, int ld, const float* __restrict__ conv_w,
                        const float* __restrict__ conv_b, int taps, const float* __restrict__ dt_bias,
                        const float* __restrict__ A_log, const float* __restrict__ skip, float* __restrict__ state,
                        long long state_stride, const int* __restrict__ slots, const int* __restrict__ cu_q,
                        float* __restrict__ y, int num_slots, int* err) {
    __shared__ __align__(16) float bs[D], cs[D];
    __shared__ float xs[DV];
    ie_pdl_trigger();
    ie_pdl_wait();
    const int head = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x;
    const int start = cu_q[seq], len = cu_q[seq + 1] - start, slot = slots[seq];
    if (len <= 0) return;
    if (slot < 0 || slot >= num_slots) {
        if (tid == 0) ie_report(err, IE_ERR_PAGE, slot, start);
        return;
    }
    const int n = at.n, p = at.p, inner = at.inner(), channels = at.channels();
    float* S = state + (size_t)slot * state_stride + (size_t)head * p * n;
    const float* tail = state + (size_t)slot * state_stride + (size_t)at.heads * p * n;
    const int sub = tid % TPC, col0 = tid / TPC;
    float s[ROUNDS][NV][4];
    const bool vec = n % 4 == 0 && state_stride % 4 == 0 && reinterpret_cast<uintptr_t>(state) % 16 == 0;
#pragma unroll
    for (int r = 0; r < ROUNDS; ++r) {
        int col = r * COLS + col0;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            int d = (i * TPC + sub) * 4;
            const float* src = S + (size_t)col * n + d;
#pragma unroll
            for (int e = 0; e < 4; ++e) s[r][i][e] = 0.f;
            if (col >= p) continue;
            if (vec) {
                if (d < n) {
                    float4 v = *reinterpret_cast<const float4*>(src);
                    s[r][i][0] = v.x; s[r][i][1] = v.y; s[r][i][2] = v.z; s[r][i][3] = v.w;
                }
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (d + e < n) s[r][i][e] = src[e];
            }
        }
    }
    const float rate = expf(A_log[head]), bias = dt_bias[head], d_skip = skip[head];
    for (int t = 0; t < len; ++t) {
        const float* row = proj + (size_t)(start + t) * ld;
        if (t > 0) __syncthreads();
        // convolved entries: D of B, D of C, DV of x (zeros beyond the sizes)
        for (int i = tid; i < 2 * D + DV; i += STEP_THREADS) {
            int c = -1;
            if (i < D) c = i < n ? at.b_at(head) + i : -1;
            else if (i < 2 * D) c = i - D < n ? at.c_at(head) + i - D : -1;
            else c = i - 2 * D < p ? at.x_at(head) + i - 2 * D : -1;
            float v = 0.f;
            if (c >= 0) {
                float acc = conv_b[c];
                for (int j = 0; j < taps; ++j) {
                    int back = taps - 1 - j;
                    float e = t - back >= 0 ? row[inner + c - (long long)back * ld] : tail[(size_t)(taps - 1 + t - back) * channels + c];
                    acc = fmaf(conv_w[(size_t)c * taps + j], e, acc);
                }
                v = bf16_round(silu_f(acc));
            }
            if (i < D) bs[i] = v;
            else if (i < 2 * D) cs[i - D] = v;
            else xs[i - 2 * D] = v;
        }
        const float dt = softplus_f(row[inner + channels + head] + bias);
        const float decay = expf(-rate * dt);
        float z[ROUNDS];
#pragma unroll
        for (int r = 0; r < ROUNDS; ++r) {
            int col = r * COLS + col0;
            z[r] = sub == 0 && col < p ? row[head * p + col] : 0.f;
        }
        __syncthreads();
        float rd[ROUNDS];
#pragma unroll
        for (int r = 0; r < ROUNDS; ++r) rd[r] = 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            int d = (i * TPC + sub) * 4;
            if (d >= D) break;
            float4 c4 = *reinterpret_cast<const float4*>(cs + d), b4 = *reinterpret_cast<const float4*>(bs + d);
#pragma unroll
            for (int r = 0; r < ROUNDS; ++r) {
                int col = r * COLS + col0;
                float u = col < DV ? dt * xs[col] : 0.f;
                s[r][i][0] = fmaf(b4.x, u, s[r][i][0] * decay);
                s[r][i][1] = fmaf(b4.y, u, s[r][i][1] * decay);
                s[r][i][2] = fmaf(b4.z, u, s[r][i][2] * decay);
                s[r][i][3] = fmaf(b4.w, u, s[r][i][3] * decay);
                rd[r] = fmaf(s[r][i][0], c4.x, rd[r]);
                rd[r] = fmaf(s[r][i][1], c4.y, rd[r]);
                rd[r] = fmaf(s[r][i][2], c4.z, rd[r]);
                rd[r] = fmaf(s[r][i][3], c4.w, rd[r]);
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
                if (col < p) y[(size_t)(start + t) * inner + head * p + col] = fmaf(d_skip, xs[col], rd[r]) * silu_f(z[r]);
            }
    }
#pragma unroll
    for (int r = 0; r < ROUNDS; ++r) {
        int col = r * COLS + col0;
        if (col >= p) continue;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            int d = (i * TPC + sub) * 4;
            float* dst = S + (size_t)col * n + d;
            if (vec) {
                if (d < n) *reinterpret_cast<float4*>(dst) = make_float4(s[r][i][0], s[r][i][1], s[r][i][2], s[r][i][3]);
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (d + e < n) dst[e] = s[r][i][e];
            }
        }
    }
}

// ---- prompt portions ---------------------------------------------------------------------------

constexpr int LDD = D + 8, LDV = DV + 8;  // rows 16 bytes longer: ldmatrix rows fall on different banks

// l[i]: the sum of the chunk's log decays up to token i (beyond the chunk's tokens: as at its last), dt[i] (beyond:
// zero).  By the block's first warp; gates: [N, heads, 3].
__device__ __forceinline__ void chunk_gates(const float* __restrict__ gates, int n0, int cnt, int head, int heads,
                                            float* l, float* dt) {
    if (threadIdx.x >= 32) return;
    int lane = threadIdx.x;
    float a[2];
#pragma unroll
    for (int k = 0; k < 2; ++k) {
        int j = lane * 2 + k;
        const float* g = gates + ((size_t)(n0 + min(j, cnt - 1)) * heads + head) * 3;
        a[k] = j < cnt ? g[2] : 0.f;
        dt[j] = j < cnt ? g[1] : 0.f;
    }
    float sum = a[0] + a[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        float v = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += v;
    }
    l[lane * 2 + 1] = sum;
    l[lane * 2] = sum - a[1];
}

// Rows of bfloat16 numbers (row j at src + j * ld) into shared rows LD entries apart, COLS entries each; rows
// beyond cnt and entries beyond `size` are zero.  `vec`: 16-byte copies are possible (and are asynchronous).
template <int THREADS, int COLS_, int LD>
__device__ __forceinline__ void bring_rows(const bf16* __restrict__ src, size_t ld, int rows, int cnt, int size, bool vec, bf16* dst) {
    if (vec) {
        for (int i = threadIdx.x; i < rows * (COLS_ / 8); i += THREADS) {
            int j = i / (COLS_ / 8), c = (i - j * (COLS_ / 8)) * 8;
            bool there = j < cnt && c < size;
            cp_async16(dst + j * LD + c, there ? src + j * ld + c : src, there);
        }
        return;
    }
    for (int i = threadIdx.x; i < rows * COLS_; i += THREADS) {
        int j = i / COLS_, c = i - j * COLS_;
        dst[j * LD + c] = (j < cnt && c < size) ? src[j * ld + c] : __float2bfloat16_rn(0.f);
    }
}

constexpr int STATE_THREADS = 256;
constexpr size_t STATE_SMEM = (size_t)CHUNK * (LDD + 2 * LDV) * sizeof(bf16);

// grid: (chunks, heads).  conv: [N, ld] bfloat16; u: [chunks, heads, p, n]; total: [chunks, heads].
__global__ void __launch_bounds__(STATE_THREADS)
chunk_state_kernel(Sizes at, const bf16* __restrict__ conv, int ld, const float* __restrict__ gates,
                   const int* __restrict__ cu_q, int num_seqs, bool vec, float* __restrict__ u, float* __restrict__ total) {
    extern __shared__ __align__(16) unsigned char raw[];
    __shared__ float l[CHUNK], dt[CHUNK];
    bf16* b_s = reinterpret_cast<bf16*>(raw);
    bf16 *x_hi = b_s + CHUNK * LDD, *x_lo = x_hi + CHUNK * LDV;
    ie_pdl_trigger();
    ie_pdl_wait();
    int seq, chunk, head = blockIdx.y;
    if (!find_chunk(cu_q, num_seqs, blockIdx.x, seq, chunk)) return;
    int start = cu_q[seq], len = cu_q[seq + 1] - start;
    int n0 = start + chunk * CHUNK, cnt = min(CHUNK, len - chunk * CHUNK);
    const bf16* rows = conv + (size_t)n0 * ld;
    bring_rows<STATE_THREADS, D, LDD>(rows + at.b_at(head), ld, CHUNK, cnt, at.n, vec, b_s);
    chunk_gates(gates, n0, cnt, head, at.heads, l, dt);
    __syncthreads();
    const float last = l[CHUNK - 1];
    if (threadIdx.x == 0) total[(size_t)blockIdx.x * at.heads + head] = expf(last);
    const bf16* x = rows + at.x_at(head);
    if (vec) {  // eight entries at a time
        for (int i = threadIdx.x; i < CHUNK * (DV / 8); i += STATE_THREADS) {
            int j = i / (DV / 8), c = (i - j * (DV / 8)) * 8;
            uint4 v = make_uint4(0u, 0u, 0u, 0u);
            if (j < cnt && c < at.p) v = *reinterpret_cast<const uint4*>(x + (size_t)j * ld + c);
            float w = expf(last - l[j]) * dt[j];
            const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&v);
            unsigned hi[4], lo[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                float2 f = __bfloat1622float2(h2[k]);
                f.x *= w; f.y *= w;
                hi[k] = pack_bf16(f.x, f.y);
                lo[k] = pack_bf16(f.x - bf16_round(f.x), f.y - bf16_round(f.y));
            }
            *reinterpret_cast<uint4*>(x_hi + j * LDV + c) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
            *reinterpret_cast<uint4*>(x_lo + j * LDV + c) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
        }
    } else {
        for (int i = threadIdx.x; i < CHUNK * DV; i += STATE_THREADS) {
            int j = i / DV, c = i - j * DV;
            float f = (j < cnt && c < at.p) ? __bfloat162float(x[(size_t)j * ld + c]) * (expf(last - l[j]) * dt[j]) : 0.f;
            bf16 h = __float2bfloat16_rn(f);
            x_hi[j * LDV + c] = h;
            x_lo[j * LDV + c] = __float2bfloat16_rn(f - __bfloat162float(h));
        }
    }
    cp_async_all();
    __syncthreads();
    int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
    float* dst = u + ((size_t)blockIdx.x * at.heads + head) * at.p * at.n;
    constexpr int WIDE = 32, NTASK = (D + WIDE - 1) / WIDE;
    for (int task = warp; task < (DV / 16) * NTASK; task += STATE_THREADS / 32) {
        int mt = task / NTASK, c0 = (task - mt * NTASK) * WIDE;
        float acc[WIDE / 8][4];
#pragma unroll
        for (int i = 0; i < WIDE / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
        for (int kk = 0; kk < CHUNK; kk += 16) {
            // A = x^T: 16 value entries x 16 tokens, from rows of tokens (transposed on the way)
            unsigned a_hi[4], a_lo[4];
            int arow = kk + (lane & 7) + ((lane >> 4) << 3), acol = mt * 16 + ((lane >> 3) & 1) * 8;
            ldsm_x4_trans(a_hi, x_hi + arow * LDV + acol);
            ldsm_x4_trans(a_lo, x_lo + arow * LDV + acol);
#pragma unroll
            for (int nt = 0; nt < WIDE / 8; nt += 2) {
                if (c0 + nt * 8 >= D) break;
                unsigned b[4];
                ldsm_x4_trans(b, b_s + (kk + (lane & 15)) * LDD + c0 + nt * 8 + (lane >> 4) * 8);
                mma_bf16(acc[nt], a_hi, b[0], b[1]);
                mma_bf16(acc[nt + 1], a_hi, b[2], b[3]);
                mma_bf16(acc[nt], a_lo, b[0], b[1]);
                mma_bf16(acc[nt + 1], a_lo, b[2], b[3]);
            }
        }
#pragma unroll
        for (int nt = 0; nt < WIDE / 8; ++nt)
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                int r = mt * 16 + g + half * 8, c = c0 + nt * 8 + t4 * 2;
                if (r >= at.p) continue;
                if (at.n % 2 == 0) {
                    if (c < at.n) *reinterpret_cast<float2*>(dst + (size_t)r * at.n + c) = make_float2(acc[nt][half * 2], acc[nt][half * 2 + 1]);
                } else {
                    if (c < at.n) dst[(size_t)r * at.n + c] = acc[nt][half * 2];
                    if (c + 1 < at.n) dst[(size_t)r * at.n + c + 1] = acc[nt][half * 2 + 1];
                }
            }
    }
}

// grid: (blocks of 256 * VEC entries, heads, requests): the state goes through a request's chunks; the state before
// each chunk is left as two bfloat16 terms, before: [chunks, heads, 2, p * n].  The next few chunks' sums are
// on their way while the last ones are added.
template <int VEC>
__global__ void __launch_bounds__(256)
chunk_scan_kernel(const float* __restrict__ u, const float* __restrict__ total, bf16* __restrict__ before,
                  float* __restrict__ state, long long state_stride, const int* __restrict__ slots,
                  const int* __restrict__ cu_q, int heads, int entries, int num_slots, int* err) {
    ie_pdl_trigger();
    ie_pdl_wait();
    int seq = blockIdx.z, head = blockIdx.y;
    int len = cu_q[seq + 1] - cu_q[seq], slot = slots[seq];
    if (len <= 0) return;
    if (slot < 0 || slot >= num_slots) {
        if (threadIdx.x == 0 && blockIdx.x == 0) ie_report(err, IE_ERR_PAGE, slot, cu_q[seq]);
        return;
    }
    int first = 0;  // the request's first chunk among the step's
    for (int i = 0; i < seq; ++i) first += (cu_q[i + 1] - cu_q[i] + CHUNK - 1) / CHUNK;
    int e = (blockIdx.x * 256 + threadIdx.x) * VEC;
    if (e >= entries) return;
    int chunks = (len + CHUNK - 1) / CHUNK;
    float* S = state + (size_t)slot * state_stride + (size_t)head * entries + e;
    const float* p = u + ((size_t)first * heads + head) * entries + e;
    const float* decay = total + (size_t)first * heads + head;
    bf16* out = before + ((size_t)first * heads + head) * 2 * entries + e;
    const size_t step = (size_t)heads * entries;
    struct alignas(4 * VEC) Pack { float v[VEC]; };
    Pack s = *reinterpret_cast<const Pack*>(S);
    constexpr int AHEAD = 8;
    Pack x[AHEAD];
    float d[AHEAD];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i)
        if (i < chunks) {
            x[i] = *reinterpret_cast<const Pack*>(p + (size_t)i * step);
            d[i] = decay[(size_t)i * heads];
        }
    for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            int c = c0 + i;
            if (c >= chunks) break;
            Pack sum = x[i];
            float a = d[i];
            if (c + AHEAD < chunks) {
                x[i] = *reinterpret_cast<const Pack*>(p + (size_t)(c + AHEAD) * step);
                d[i] = decay[(size_t)(c + AHEAD) * heads];
            }
            bf16* dst = out + (size_t)c * 2 * step;
            struct alignas(2 * VEC) Half { bf16 v[VEC]; } hi, lo;
#pragma unroll
            for (int v = 0; v < VEC; ++v) {
                hi.v[v] = __float2bfloat16_rn(s.v[v]);
                lo.v[v] = __float2bfloat16_rn(s.v[v] - __bfloat162float(hi.v[v]));
                s.v[v] = fmaf(a, s.v[v], sum.v[v]);
            }
            *reinterpret_cast<Half*>(dst) = hi;
            *reinterpret_cast<Half*>(dst + entries) = lo;
        }
    }
    *reinterpret_cast<Pack*>(S) = s;
}

// eight warps: warp w takes the sixteen rows (w & 3) * 16 .. and one half of the value entries
constexpr int OUT_THREADS = 256;
constexpr int PAIRS = DV / 16, WARP_PAIRS = (PAIRS + 1) / 2, TILES = 2 * WARP_PAIRS;  // of sixteen value entries; of eight
constexpr size_t OUT_SMEM = (size_t)(2 * CHUNK * LDD + 2 * DV * LDD + CHUNK * LDV) * sizeof(bf16);

// grid: (chunks, heads).  before: the state before each chunk as two terms; proj: for z; y: [N, heads * p].
__global__ void __launch_bounds__(OUT_THREADS)
chunk_out_kernel(Sizes at, const bf16* __restrict__ conv, int ld, const float* __restrict__ gates,
                 const bf16* __restrict__ before, const float* __restrict__ proj, int proj_ld,
                 const float* __restrict__ skip, const int* __restrict__ cu_q, int num_seqs, bool vec, bool pairs,
                 float* __restrict__ y) {
    extern __shared__ __align__(16) unsigned char raw[];
    __shared__ float l[CHUNK], dt[CHUNK];
    bf16* c_s = reinterpret_cast<bf16*>(raw);
    bf16 *b_s = c_s + CHUNK * LDD, *s_hi = b_s + CHUNK * LDD, *s_lo = s_hi + DV * LDD, *x_s = s_lo + DV * LDD;
    ie_pdl_trigger();
    ie_pdl_wait();
    int seq, chunk, head = blockIdx.y;
    if (!find_chunk(cu_q, num_seqs, blockIdx.x, seq, chunk)) return;
    int start = cu_q[seq], len = cu_q[seq + 1] - start;
    int n0 = start + chunk * CHUNK, cnt = min(CHUNK, len - chunk * CHUNK);
    const bf16* rows = conv + (size_t)n0 * ld;
    const bf16* S = before + ((size_t)blockIdx.x * at.heads + head) * 2 * at.p * at.n;
    bring_rows<OUT_THREADS, D, LDD>(rows + at.c_at(head), ld, CHUNK, cnt, at.n, vec, c_s);
    bring_rows<OUT_THREADS, D, LDD>(S, at.n, DV, at.p, at.n, vec, s_hi);
    bring_rows<OUT_THREADS, D, LDD>(S + (size_t)at.p * at.n, at.n, DV, at.p, at.n, vec, s_lo);
    bring_rows<OUT_THREADS, D, LDD>(rows + at.b_at(head), ld, CHUNK, cnt, at.n, vec, b_s);
    bring_rows<OUT_THREADS, DV, LDV>(rows + at.x_at(head), ld, CHUNK, cnt, at.p, vec, x_s);
    chunk_gates(gates, n0, cnt, head, at.heads, l, dt);
    cp_async_all();
    __syncthreads();
    int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
    const int wr = warp & 3, wc = warp >> 2, col0 = wc * WARP_PAIRS * 16;  // the warp's rows and first value entry
    if (wr * 16 >= cnt || col0 >= DV) return;
    float o[TILES][4];
#pragma unroll
    for (int i = 0; i < TILES; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    const int arow = (wr * 16 + (lane & 15)) * LDD + (lane >> 4) * 8;  // a warp's 16 rows of C
    const int brow = (lane & 7) + ((lane >> 4) << 3), bcol = ((lane >> 3) & 1) * 8;
    // what the state before the chunk holds: exp(l_i) S^T C_i
#pragma unroll 2
    for (int kk = 0; kk < D; kk += 16) {
        unsigned a[4];
        ldsm_x4(a, c_s + arow + kk);
#pragma unroll
        for (int nt = 0; nt < TILES; nt += 2) {
            if (col0 + nt * 8 >= DV) break;
            unsigned b_hi[4], b_lo[4];
            ldsm_x4(b_hi, s_hi + (col0 + nt * 8 + brow) * LDD + kk + bcol);
            ldsm_x4(b_lo, s_lo + (col0 + nt * 8 + brow) * LDD + kk + bcol);
            mma_bf16(o[nt], a, b_hi[0], b_hi[1]);
            mma_bf16(o[nt + 1], a, b_hi[2], b_hi[3]);
            mma_bf16(o[nt], a, b_lo[0], b_lo[1]);
            mma_bf16(o[nt + 1], a, b_lo[2], b_lo[3]);
        }
    }
    const int r_a = wr * 16 + g, r_b = r_a + 8;
    const float l_a = l[r_a], l_b = l[r_b];
    {
        float f_a = expf(l_a), f_b = expf(l_b);
#pragma unroll
        for (int i = 0; i < TILES; ++i) { o[i][0] *= f_a; o[i][1] *= f_a; o[i][2] *= f_b; o[i][3] *= f_b; }
    }
    // sixteen tokens at a time, up to the warp's last row
    for (int kt = 0; kt <= wr; ++kt) {
        float s[2][4];
#pragma unroll
        for (int i = 0; i < 2; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
#pragma unroll 4
        for (int kk = 0; kk < D; kk += 16) {
            unsigned a[4], b[4];
            ldsm_x4(a, c_s + arow + kk);
            ldsm_x4(b, b_s + (kt * 16 + brow) * LDD + kk + bcol);
            mma_bf16(s[0], a, b[0], b[1]);
            mma_bf16(s[1], a, b[2], b[3]);
        }
        unsigned p_hi[4], p_lo[4];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            float w[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                int j = kt * 16 + i * 8 + t4 * 2 + (e & 1), r = e < 2 ? r_a : r_b;
                w[e] = j <= r ? s[i][e] * (expf((e < 2 ? l_a : l_b) - l[j]) * dt[j]) : 0.f;
            }
            p_hi[i * 2] = pack_bf16(w[0], w[1]);
            p_hi[i * 2 + 1] = pack_bf16(w[2], w[3]);
            p_lo[i * 2] = pack_bf16(w[0] - bf16_round(w[0]), w[1] - bf16_round(w[1]));
            p_lo[i * 2 + 1] = pack_bf16(w[2] - bf16_round(w[2]), w[3] - bf16_round(w[3]));
        }
#pragma unroll
        for (int nt = 0; nt < TILES; nt += 2) {
            if (col0 + nt * 8 >= DV) break;
            unsigned b[4];
            ldsm_x4_trans(b, x_s + (kt * 16 + (lane & 15)) * LDV + col0 + nt * 8 + (lane >> 4) * 8);
            mma_bf16(o[nt], p_hi, b[0], b[1]);
            mma_bf16(o[nt + 1], p_hi, b[2], b[3]);
            mma_bf16(o[nt], p_lo, b[0], b[1]);
            mma_bf16(o[nt + 1], p_lo, b[2], b[3]);
        }
    }
    // skip, gate, write
    const float d_skip = skip[head];
    const int inner = at.inner();
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        int r = half ? r_b : r_a;
        if (r >= cnt) continue;
        const float* z = proj + (size_t)(n0 + r) * proj_ld + (size_t)head * at.p;
        float* dst = y + (size_t)(n0 + r) * inner + (size_t)head * at.p;
#pragma unroll
        for (int i = 0; i < TILES; ++i) {
            int c = col0 + i * 8 + t4 * 2;
            if (pairs) {
                if (c >= at.p) break;
                float2 z2 = *reinterpret_cast<const float2*>(z + c);
                float2 x2 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(x_s + r * LDV + c));
                *reinterpret_cast<float2*>(dst + c) = make_float2(fmaf(d_skip, x2.x, o[i][half * 2]) * silu_f(z2.x),
                                                                  fmaf(d_skip, x2.y, o[i][half * 2 + 1]) * silu_f(z2.y));
                continue;
            }
#pragma unroll
            for (int e = 0; e < 2; ++e)
                if (c + e < at.p)
                    dst[c + e] = fmaf(d_skip, __bfloat162float(x_s[r * LDV + c + e]), o[i][half * 2 + e]) * silu_f(z[c + e]);
        }
    }
}
}  // namespace

IE_API int ie_state_space_dims(int* n, int* p) {
    *n = D;
    *p = DV;
    return CHUNK;
}

// Requests of at most 8 tokens each.  proj: at the z columns; state: [slots][heads * p * n, then the kept inputs].
IE_API int ie_state_space_step(const float* proj, int ld, int heads, int groups, int n, int p, const float* conv_w,
                               const float* conv_b, int taps, const float* dt_bias, const float* A_log,
                               const float* skip, float* state, long long state_stride, const int* slots,
                               const int* cu_q, int num_seqs, int max_q_len, float* y, int num_slots, int* err,
                               void* stream) {
    if (num_seqs <= 0) return 0;
    if (n < 1 || p < 1 || n > D || p > DV || heads < 1 || groups < 1 || heads % groups || taps < 1 || max_q_len > STEP_MOST)
        return (int)cudaErrorInvalidValue;
    return ie_launch(state_space_step_kernel, dim3(heads, num_seqs), dim3(STEP_THREADS), 0, (cudaStream_t)stream,
                     Sizes{heads, groups, n, p}, proj, ld, conv_w, conv_b, taps, dt_bias, A_log, skip, state,
                     state_stride, slots, cu_q, y, num_slots, err);
}

// chunks: at least as many chunks of 64 tokens as the step's requests have; u: [chunks, heads, p * n] floats, total:
// [chunks, heads] floats, before: [chunks, heads, 2, p * n] bfloat16.  conv: the convolved rows, bfloat16, `ld` apart.
IE_API int ie_state_space_chunks(const void* conv, int ld, const float* gates, int heads, int groups, int n, int p,
                                 const float* proj, int proj_ld, const float* skip, float* state,
                                 long long state_stride, const int* slots, const int* cu_q, int num_seqs, int chunks,
                                 float* u, float* total, void* before, float* y, int num_slots, int* err, void* stream) {
    if (num_seqs <= 0 || chunks <= 0) return 0;
    if (n < 1 || p < 1 || n > D || p > DV || heads < 1 || groups < 1 || heads % groups || ld < heads * p + 2 * groups * n)
        return (int)cudaErrorInvalidValue;
    cudaStream_t s = (cudaStream_t)stream;
    static IePerDevice allowed_state, allowed_out;
    cudaError_t e = ie_allow_smem(allowed_state, chunk_state_kernel, STATE_SMEM);
    if (e == cudaSuccess) e = ie_allow_smem(allowed_out, chunk_out_kernel, OUT_SMEM);
    if (e != cudaSuccess) return (int)e;
    const Sizes at{heads, groups, n, p};
    const bool vec = n % 8 == 0 && p % 8 == 0 && ld % 8 == 0 &&
                     ((reinterpret_cast<uintptr_t>(conv) | reinterpret_cast<uintptr_t>(before)) % 16 == 0);
    const bool pairs = p % 2 == 0 && proj_ld % 2 == 0 &&
                       ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(y)) % 8 == 0);
    int rc = ie_launch(chunk_state_kernel, dim3(chunks, heads), dim3(STATE_THREADS), STATE_SMEM, s, at, (const bf16*)conv,
                       ld, gates, cu_q, num_seqs, vec, u, total);
    if (rc != 0) return rc;
    int entries = n * p;
    if (entries % 4 == 0 && state_stride % 4 == 0 &&
        ((reinterpret_cast<uintptr_t>(state) | reinterpret_cast<uintptr_t>(u) | reinterpret_cast<uintptr_t>(before)) % 16 == 0))
        rc = ie_launch(chunk_scan_kernel<4>, dim3((entries + 1023) / 1024, heads, num_seqs), dim3(256), 0, s,
                       (const float*)u, (const float*)total, (bf16*)before, state, state_stride, slots, cu_q, heads,
                       entries, num_slots, err);
    else
        rc = ie_launch(chunk_scan_kernel<1>, dim3((entries + 255) / 256, heads, num_seqs), dim3(256), 0, s,
                       (const float*)u, (const float*)total, (bf16*)before, state, state_stride, slots, cu_q, heads,
                       entries, num_slots, err);
    if (rc != 0) return rc;
    return ie_launch(chunk_out_kernel, dim3(chunks, heads), dim3(OUT_THREADS), OUT_SMEM, s, at, (const bf16*)conv, ld,
                     gates, (const bf16*)before, proj, proj_ld, skip, cu_q, num_seqs, vec, pairs, y);
}
