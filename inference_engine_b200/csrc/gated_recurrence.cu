// Kernels of recurrent mixers whose state is a matrix per head that decays and takes an outer
// product per token:   S_t = diag(a_t) S_(t-1) + w_t u_t^T,   o_t = S_t^T q_t,
// with S of dim x cols (32-bit, kept column by column in the request's state slot).
//
//  * gated-write linear attention (HGRN2): a_t = f_t and w_t = 1 - f_t per head and channel,
//    u_t = v_t, f_t = lower + (1 - lower) * sigmoid(. + bias); q_t = silu(.).
//  * matrix memory with exponential gates (mLSTM): a_t and a write gate b_t are one number per
//    head, w_t = k_t, u_t = b_t v_t, and one more column whose value is 1 carries the
//    normaliser n_t = a_t n_(t-1) + b_t k_t.  The gates come from a running maximum m_t that
//    starts at 0:  m_t = max(logf_t + m_(t-1), logi_t),  a_t = exp(logf_t + m_(t-1) - m_t),
//    b_t = exp(logi_t - m_t);  o_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + 1e-6).
//
//  * gated linear attention: a_t per head and channel from a low-rank map of the input,
//    a_t = sigmoid(z_t)^(1 / tau) with z_t = W2 y_t + b (y_t the input's projection to a few
//    numbers), taken as exp(logsigmoid(z_t) / tau); w_t = k_t, u_t = v_t; the read-out's gate is
//    silu(.) instead of sigmoid(.).
//
//  * retention: a_t is one constant per head and the write gate is 1 (the gates' array then holds one
//    token's numbers for all of them: a token stride of 0), w_t = k_t, u_t = v_t with q and k rotated by
//    position; the read-out's unit root mean square has no weight.
//
//  * state-space duality (Mamba-2): a_t = exp(-exp(A_log) dt_t) and the write gate dt_t are one number per head,
//    dt_t = softplus(. + dt_bias); w_t = B_t and q_t = C_t belong to groups of heads (`heads_per_unit` heads read the
//    same rows of q and w), u_t = dt_t x_t; x, B and C come from a short convolution with a bias and silu.
//    y_t = S_t^T C_t + D x_t, times silu(z_t), then divided by its root mean square in equal parts of the row.
//
// Kernels: conv_silu (the convolution over the step's tokens and, before them, the slot's kept inputs; a thread
// takes a channel through sixteen tokens) with the heads' gates in the same launch; gated_group_norm (skip, gate, norm in parts,
// weight; it also moves the slot's kept convolution inputs on, which no earlier kernel of the step may do); rotate_heads (in place in the 32-bit projection: the first rot_dims entries of every head, by
// pairs (i, i + rot_dims / 2), from the 32-bit table of angles); lowrank_decay (a block takes sixteen tokens and 128 channels, so that a row of W2 is read
// once per sixteen tokens); short_conv_residual (+ tail update): out = x + causal convolution of x over time per
// channel, the last taps - 1 inputs kept per request; hgrn2_gates; mlstm_gates (a warp per request
// and head walks the step's tokens in order); gated_recurrence (columns of S do not interact: a
// block owns some columns of one head of one request, TPC lanes a column, tokens in order, eight at
// a time through a ring of four shared-memory buffers, three chunks on their way); recurrence_readout (normaliser,
// unit root mean square per head, weight, output gate).  Every sum is taken in an order that
// depends on the sizes alone, never on how a request's tokens were cut into steps or batched.
#include "common.cuh"
#include <math.h>

namespace {

__device__ __forceinline__ float silu_f(float y) { return y / (1.0f + expf(-y)); }
__device__ __forceinline__ float sigmoid_f(float y) { return 1.0f / (1.0f + expf(-y)); }
__device__ __forceinline__ float logsigmoid_f(float y) { return fminf(y, 0.f) - log1pf(expf(-fabsf(y))); }

// grid: (tokens, blocks of channels).  x and out: [N, channels] in the compute dtype; w: [channels, taps], the last tap
// weighs the token itself; tail: the slot's kept inputs [taps - 1][channels], oldest first.
template <typename T>
__global__ void __launch_bounds__(256)
short_conv_residual_kernel(const T* __restrict__ x, const float* __restrict__ w, const float* __restrict__ state,
                           long long state_stride, const int* __restrict__ slots,
                           const int* __restrict__ seq_of_token, const int* __restrict__ cu_q,
                           T* __restrict__ out, int channels, int taps, int num_slots, int* err) {
    ie_pdl_trigger();
    ie_pdl_wait();
    int n = blockIdx.x;
    int seq = seq_of_token[n];
    int t = n - cu_q[seq];
    int slot = slots[seq];
    if (slot < 0 || slot >= num_slots) {
        if (threadIdx.x == 0) ie_report(err, IE_ERR_PAGE, slot, n);
        return;
    }
    const float* tail = state + (size_t)slot * state_stride;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < channels; c += gridDim.y * blockDim.x) {
        float acc = 0.f;
        for (int j = 0; j < taps; ++j) {
            int back = taps - 1 - j;
            float xv = (t - back >= 0) ? ie_load(x + (size_t)(n - back) * channels + c)
                                       : tail[(size_t)(taps - 1 + t - back) * channels + c];
            acc = fmaf(w[(size_t)c * taps + j], xv, acc);
        }
        ie_store(out + (size_t)n * channels + c, ie_load(x + (size_t)n * channels + c) + acc);
    }
}

// grid: (requests of the step, blocks of channels): the kept inputs become the last taps - 1 of (kept, new).
template <typename T>
__global__ void short_conv_tail_kernel(const T* __restrict__ x, float* __restrict__ state, long long state_stride,
                                       const int* __restrict__ slots, const int* __restrict__ cu_q, int channels,
                                       int taps, int num_slots) {
    ie_pdl_trigger();
    ie_pdl_wait();
    int seq = blockIdx.x;
    int start = cu_q[seq], len = cu_q[seq + 1] - start;
    int slot = slots[seq];
    if (len <= 0 || slot < 0 || slot >= num_slots) return;
    float* tail = state + (size_t)slot * state_stride;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < channels; c += gridDim.y * blockDim.x) {
        // a thread owns a channel and goes through the rows in rising order, so a kept row is
        // read before it is overwritten
        for (int j = 0; j < taps - 1; ++j) {
            int tt = len - (taps - 1) + j;
            float xv = tt >= 0 ? ie_load(x + (size_t)(start + tt) * channels + c)
                               : tail[(size_t)(taps - 1 + tt) * channels + c];
            tail[(size_t)j * channels + c] = xv;
        }
    }
}

// proj: [N, ld] 32-bit, columns q (size), forget pre-activations (size), then whatever follows.
// In place: q <- silu(q), f <- lower + (1 - lower) * sigmoid(f + bias); write[n, c] = 1 - f.
__global__ void hgrn2_gates_kernel(float* __restrict__ proj, int ld, const float* __restrict__ bias,
                                   const float* __restrict__ lower, float* __restrict__ write, int size,
                                   size_t total) {
    ie_pdl_trigger();
    ie_pdl_wait();
    size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    size_t stride = (size_t)gridDim.x * blockDim.x;
    for (; idx < total; idx += stride) {
        size_t n = idx / size;
        int c = (int)(idx - n * size);
        float* row = proj + n * ld;
        row[c] = silu_f(row[c]);
        float l = lower[c];
        float f = l + (1.0f - l) * sigmoid_f(row[size + c] + bias[c]);
        row[size + c] = f;
        write[idx] = 1.0f - f;
    }
}

// grid: (tokens, blocks of pairs).  x: `units` heads of `dim` entries at the start of rows `ld` apart.
__global__ void __launch_bounds__(128)
rotate_heads_kernel(float* __restrict__ x, int ld, const int* __restrict__ positions, const float* __restrict__ table,
                    int rot_dims, int table_positions, int units, int dim, int* err) {
    ie_pdl_trigger();
    ie_pdl_wait();
    int n = blockIdx.x, half = rot_dims / 2;
    int pos = positions[n];
    if (pos < 0 || pos >= table_positions) {
        if (threadIdx.x == 0) ie_report(err, IE_ERR_POSITION, pos, n);
        return;
    }
    const float* cs = table + (size_t)pos * rot_dims;  // cos of the angles, then their sin
    for (int i = blockIdx.y * 128 + threadIdx.x; i < units * half; i += gridDim.y * 128) {
        int unit = i / half, j = i - unit * half;
        float* p = x + (size_t)n * ld + (size_t)unit * dim + j;
        float u = p[0], v = p[half], c = cs[j], s = cs[half + j];
        p[0] = u * c - v * s;
        p[half] = v * c + u * s;
    }
}

// grid: (heads, requests), one warp each.  gi, gf: the gates' pre-activations, element (n, head) at
// [n * ld + head].  gates: [N, heads, 3] = (a, b, exp(-m)).  m: the running maximum of a head,
// in the slot at `m_offset + head`.
__global__ void __launch_bounds__(32)
mlstm_gates_kernel(const float* __restrict__ gi, const float* __restrict__ gf, int ld,
                   const float* __restrict__ bias_i, const float* __restrict__ bias_f, float cap,
                   float* __restrict__ state, long long state_stride, long long m_offset,
                   const int* __restrict__ slots, const int* __restrict__ cu_q, float* __restrict__ gates,
                   int heads, int num_slots) {
    ie_pdl_trigger();
    ie_pdl_wait();
    int head = blockIdx.x, seq = blockIdx.y, lane = threadIdx.x;
    int start = cu_q[seq], len = cu_q[seq + 1] - start;
    int slot = slots[seq];
    if (len <= 0 || slot < 0 || slot >= num_slots) return;
    float* m_ptr = state + (size_t)slot * state_stride + m_offset + head;
    float m = *m_ptr;
    float bi = bias_i[head], bf = bias_f[head];
    for (int t0 = 0; t0 < len; t0 += 32) {
        int cnt = min(32, len - t0);
        float li = 0.f, lf = 0.f;
        if (lane < cnt) {
            size_t n = (size_t)(start + t0 + lane);
            li = cap * tanhf((gi[n * ld + head] + bi) / cap);
            lf = logsigmoid_f(cap * tanhf((gf[n * ld + head] + bf) / cap));
        }
        float m_before = 0.f, m_mine = 0.f;
        for (int j = 0; j < cnt; ++j) {  // the chain, the same in every lane
            float fj = __shfl_sync(0xffffffffu, lf, j), ij = __shfl_sync(0xffffffffu, li, j);
            float m_new = fmaxf(fj + m, ij);
            if (lane == j) { m_before = m; m_mine = m_new; }
            m = m_new;
        }
        if (lane < cnt) {
            float* g = gates + ((size_t)(start + t0 + lane) * heads + head) * 3;
            g[0] = expf(lf + m_before - m_mine);
            g[1] = expf(li - m_mine);
            g[2] = expf(-m_mine);
        }
    }
    if (lane == 0) *m_ptr = m;
}

// grid: (blocks of LD_TOKENS tokens, blocks of 128 channels).  y: element (n, r) at [n * y_ld + r]; w2: [channels, rank];
// decay: [N, channels] = exp(logsigmoid(w2 y + bias) * inv_tau).  A channel's sum runs over r in rising order.
// The block's 128 rows of w2 and its tokens' inputs pass through shared memory 32 ranks at a time: a warp
// reads 32 consecutive numbers of a row at once, and rows sit 33 words apart so that the threads of a
// warp, one channel each, read different banks.
constexpr int LD_TOKENS = 16, LD_RANKS = 32;
__global__ void __launch_bounds__(128)
lowrank_decay_kernel(const float* __restrict__ y, int y_ld, const float* __restrict__ w2,
                     const float* __restrict__ bias, float inv_tau, float* __restrict__ decay, int num_tokens,
                     int channels, int rank) {
    __shared__ float ws[128 * (LD_RANKS + 1)];
    __shared__ float ys[LD_TOKENS * LD_RANKS];
    ie_pdl_trigger();
    ie_pdl_wait();
    int n0 = blockIdx.x * LD_TOKENS, c0 = blockIdx.y * 128;
    int cnt = min(LD_TOKENS, num_tokens - n0);
    int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float acc[LD_TOKENS];
#pragma unroll
    for (int t = 0; t < LD_TOKENS; ++t) acc[t] = 0.f;
    for (int r0 = 0; r0 < rank; r0 += LD_RANKS) {
        int width = min(LD_RANKS, rank - r0);
        if (r0 > 0) __syncthreads();  // everyone is done with the last piece
        for (int row = warp; row < 128; row += 4) {
            int c = c0 + row;
            ws[row * (LD_RANKS + 1) + lane] = (c < channels && lane < width) ? w2[(size_t)c * rank + r0 + lane] : 0.f;
        }
        for (int t = warp; t < LD_TOKENS; t += 4)
            ys[t * LD_RANKS + lane] = (t < cnt && lane < width) ? y[(size_t)(n0 + t) * y_ld + r0 + lane] : 0.f;
        __syncthreads();
        const float* wrow = ws + threadIdx.x * (LD_RANKS + 1);
        for (int r = 0; r < width; ++r) {
            float wv = wrow[r];
#pragma unroll
            for (int t = 0; t < LD_TOKENS; ++t) acc[t] = fmaf(wv, ys[t * LD_RANKS + r], acc[t]);
        }
    }
    int c = c0 + threadIdx.x;
    if (c >= channels) return;
    float b = bias != nullptr ? bias[c] : 0.f;
#pragma unroll
    for (int t = 0; t < LD_TOKENS; ++t)
        if (t < cnt) decay[(size_t)(n0 + t) * channels + c] = expf(logsigmoid_f(acc[t] + b) * inv_tau);
}

// The short convolution with bias and silu of a 32-bit projection, and the state-space heads' gates.
// grid: (blocks of CS_TOKENS tokens, blocks of 128 channels, + 1 for the gates).  x: [N, x_ld] 32-bit; w: [channels,
// taps], the last tap weighs the token itself; tail: the slot's kept inputs [taps - 1][channels], oldest first, at
// `tail_at` of the slot; out: [N, out_ld].  TAPS 0: any number of taps, each fetched anew.
// gates: [N, heads, 3] = (exp(-exp(A_log) dt), dt, -exp(A_log) dt), dt = softplus(dt_pre + dt_bias).
constexpr int CS_TOKENS = 16;
__device__ __forceinline__ float softplus_f(float y) { return y > 20.0f ? y : log1pf(expf(y)); }

template <typename T, int TAPS>
__global__ void __launch_bounds__(128)
conv_silu_kernel(const float* __restrict__ x, int x_ld, const float* __restrict__ w, const float* __restrict__ bias,
                 const float* __restrict__ state, long long state_stride, long long tail_at,
                 const int* __restrict__ slots, const int* __restrict__ seq_of_token, const int* __restrict__ cu_q,
                 T* __restrict__ out, int out_ld, int num_tokens, int channels, int taps, int num_slots,
                 const float* __restrict__ dt_pre, const float* __restrict__ dt_bias, const float* __restrict__ A_log,
                 float* __restrict__ gates, int heads, int* err) {
    ie_pdl_trigger();
    ie_pdl_wait();
    const int n0 = blockIdx.x * CS_TOKENS, n1 = min(n0 + CS_TOKENS, num_tokens);
    if (blockIdx.y + 1 == gridDim.y) {
        for (int i = threadIdx.x; i < (n1 - n0) * heads; i += blockDim.x) {
            int r = i / heads, h = i - r * heads;
            size_t n = (size_t)(n0 + r);
            float dt = softplus_f(dt_pre[n * x_ld + h] + dt_bias[h]);
            float a = -expf(A_log[h]) * dt;
            float* g = gates + (n * heads + h) * 3;
            g[0] = expf(a);
            g[1] = dt;
            g[2] = a;
        }
        return;
    }
    const int c = blockIdx.y * 128 + threadIdx.x;
    const bool live = c < channels;
    const float b = live && bias != nullptr ? bias[c] : 0.f;
    constexpr int KEEP = TAPS > 1 ? TAPS - 1 : 1;
    float wt[TAPS > 0 ? TAPS : 1], before[KEEP];  // before[i]: the input i + 1 tokens back
#pragma unroll
    for (int j = 0; j < TAPS; ++j) wt[j] = live ? w[(size_t)c * taps + j] : 0.f;
    int seq = -1, first = 0, slot = -1;
    const float* tail = nullptr;
    for (int n = n0; n < n1; ++n) {
        int s = seq_of_token[n];
        bool fresh = s != seq;
        if (fresh) {
            seq = s;
            first = cu_q[seq];
            slot = slots[seq];
            if (slot < 0 || slot >= num_slots) {
                if (threadIdx.x == 0) ie_report(err, IE_ERR_PAGE, slot, n);
                return;
            }
            tail = state + (size_t)slot * state_stride + tail_at;
        }
        if (!live) continue;
        if (TAPS > 0 && n == n0 && n1 - n0 == CS_TOKENS && n1 <= cu_q[seq + 1]) {
            // a whole tile of one request: every input is on its way before the first is used
            float in[CS_TOKENS + KEEP];
#pragma unroll
            for (int i = 0; i < CS_TOKENS; ++i) in[KEEP + i] = x[(size_t)(n0 + i) * x_ld + c];
#pragma unroll
            for (int i = 0; i < TAPS - 1; ++i) {
                int back = TAPS - 1 - i;
                in[i] = n0 - back >= first ? x[(size_t)(n0 - back) * x_ld + c] : tail[(size_t)(taps - 1 + n0 - first - back) * channels + c];
            }
#pragma unroll
            for (int i = 0; i < CS_TOKENS; ++i) {
                float acc = b;
#pragma unroll
                for (int j = 0; j < TAPS; ++j) acc = fmaf(wt[j], in[KEEP + i - (TAPS - 1) + j], acc);
                ie_store(out + (size_t)(n0 + i) * out_ld + c, silu_f(acc));
            }
            return;
        }
        const int t = n - first;
        auto earlier = [&](int back) {
            return t - back >= 0 ? x[(size_t)(n - back) * x_ld + c] : tail[(size_t)(taps - 1 + t - back) * channels + c];
        };
        float acc = b, own = x[(size_t)n * x_ld + c];
        if (TAPS > 0) {
            if (fresh)
#pragma unroll
                for (int i = 0; i < TAPS - 1; ++i) before[i] = earlier(i + 1);
#pragma unroll
            for (int j = 0; j < TAPS - 1; ++j) acc = fmaf(wt[j], before[TAPS - 2 - j], acc);
            acc = fmaf(wt[TAPS > 0 ? TAPS - 1 : 0], own, acc);
#pragma unroll
            for (int i = KEEP - 1; i > 0; --i) before[i] = before[i - 1];
            before[0] = own;
        } else {
            for (int j = 0; j < taps - 1; ++j) acc = fmaf(w[(size_t)c * taps + j], earlier(taps - 1 - j), acc);
            acc = fmaf(w[(size_t)c * taps + taps - 1], own, acc);
        }
        ie_store(out + (size_t)n * out_ld + c, silu_f(acc));
    }
}

// The slot's kept convolution inputs moved on by the step's tokens: the last taps - 1 of (kept, new).  A thread owns
// a channel; every value is read before the first is written.
__device__ __forceinline__ void move_kept_inputs(int seq, int c, const float* __restrict__ raw, int raw_ld,
                                                 float* __restrict__ state, long long state_stride, long long tail_at,
                                                 const int* __restrict__ slots, const int* __restrict__ cu_q, int channels,
                                                 int taps, int num_slots) {
    const int start = cu_q[seq], len = cu_q[seq + 1] - start, slot = slots[seq];
    if (c >= channels || len <= 0 || slot < 0 || slot >= num_slots) return;
    float* tail = state + (size_t)slot * state_stride + tail_at + c;
    auto kept = [&](int j) {
        int tt = len - (taps - 1) + j;
        return tt >= 0 ? raw[(size_t)(start + tt) * raw_ld + c] : tail[(size_t)(taps - 1 + tt) * channels];
    };
    constexpr int MOST = 3;
    if (taps - 1 <= MOST) {
        float v[MOST];
#pragma unroll
        for (int j = 0; j < MOST; ++j)
            if (j < taps - 1) v[j] = kept(j);
#pragma unroll
        for (int j = 0; j < MOST; ++j)
            if (j < taps - 1) tail[(size_t)j * channels] = v[j];
        return;
    }
    for (int j = 0; j < taps - 1; ++j) tail[(size_t)j * channels] = kept(j);  // (rising: read before it is overwritten)
}

// grid: tokens * parts, then the blocks that move the kept inputs (256 channels of a request each).  y: [N, size] 32-bit; with `x` (the convolved values, [N, x_ld]) D[head] x is added, and
// with `z` ([N, z_ld] 32-bit) the sum is multiplied by silu(z); then each of the row's equal parts is divided by
// its root mean square and multiplied by the weight.  raw: the convolution's inputs, [N, raw_ld] 32-bit.
// VEC: y alone (no x, no z), four entries at a time, a part of at most GN_THREADS * 16 entries.
constexpr int GN_THREADS = 256;
template <typename T, bool VEC>
__global__ void __launch_bounds__(GN_THREADS)
gated_group_norm_kernel(const float* __restrict__ y, const float* __restrict__ x, int x_ld, const float* __restrict__ skip,
                        const float* __restrict__ z, int z_ld, const float* __restrict__ weight, float eps,
                        T* __restrict__ out, int out_ld, int num_tokens, int size, int parts, int vdim,
                        const float* __restrict__ raw, int raw_ld, float* __restrict__ state, long long state_stride,
                        long long tail_at, const int* __restrict__ slots, const int* __restrict__ cu_q, int channels,
                        int taps, int num_slots) {
    extern __shared__ __align__(16) float part_buf[];  // [size / parts]
    __shared__ float red[GN_THREADS / 32];
    ie_pdl_trigger();
    if ((int)blockIdx.x >= num_tokens * parts) {
        ie_pdl_wait();
        int i = blockIdx.x - num_tokens * parts, per = (channels + GN_THREADS - 1) / GN_THREADS;
        move_kept_inputs(i / per, (i % per) * GN_THREADS + threadIdx.x, raw, raw_ld, state, state_stride, tail_at, slots, cu_q,
                         channels, taps, num_slots);
        return;
    }
    const int n = blockIdx.x / parts, part = blockIdx.x - n * parts, width = size / parts, at = part * width;
    const float* yr = y + (size_t)n * size + at;
    constexpr int PIECES = 4;
    float4 w4[PIECES], y4[PIECES];
    float ss = 0.f;
    if constexpr (VEC) {
#pragma unroll
        for (int i = 0; i < PIECES; ++i) {  // (no kernel writes the weight)
            int c = (i * GN_THREADS + threadIdx.x) * 4;
            if (c < width) w4[i] = *reinterpret_cast<const float4*>(weight + at + c);
        }
        ie_pdl_wait();
#pragma unroll
        for (int i = 0; i < PIECES; ++i) {
            int c = (i * GN_THREADS + threadIdx.x) * 4;
            y4[i] = c < width ? *reinterpret_cast<const float4*>(yr + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int i = 0; i < PIECES; ++i)
            ss = fmaf(y4[i].x, y4[i].x, fmaf(y4[i].y, y4[i].y, fmaf(y4[i].z, y4[i].z, fmaf(y4[i].w, y4[i].w, ss))));
    } else {
        ie_pdl_wait();
        for (int i = threadIdx.x; i < width; i += GN_THREADS) {
            float v = yr[i];
            if (x != nullptr) v = fmaf(skip[(at + i) / vdim], x[(size_t)n * x_ld + at + i], v);
            if (z != nullptr) v *= silu_f(z[(size_t)n * z_ld + at + i]);
            part_buf[i] = v;
            ss = fmaf(v, v, ss);
        }
    }
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    float total = 0.f;
#pragma unroll
    for (int w = 0; w < GN_THREADS / 32; ++w) total += red[w];
    const float inv = 1.0f / sqrtf(total / (float)width + eps);
    T* dst = out + (size_t)n * out_ld + at;
    if constexpr (VEC) {
#pragma unroll
        for (int i = 0; i < PIECES; ++i) {
            int c = (i * GN_THREADS + threadIdx.x) * 4;
            if (c >= width) break;
            float4 v = make_float4(y4[i].x * inv * w4[i].x, y4[i].y * inv * w4[i].y, y4[i].z * inv * w4[i].z, y4[i].w * inv * w4[i].w);
            if constexpr (sizeof(T) == 2) {
                __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
                *reinterpret_cast<uint2*>(dst + c) = make_uint2(*reinterpret_cast<unsigned*>(&lo), *reinterpret_cast<unsigned*>(&hi));
            } else {
                *reinterpret_cast<float4*>(dst + c) = v;
            }
        }
    } else {
        for (int i = threadIdx.x; i < width; i += GN_THREADS) ie_store(dst + i, part_buf[i] * inv * weight[at + i]);
    }
}

constexpr int GR_THREADS = 128;
constexpr int GR_CHUNK = 8;  // tokens staged in shared memory at a time
constexpr int GR_STAGES = 4;  // ... in a ring of so many buffers: three chunks are on their way while one is worked on

__device__ __forceinline__ void cp_async4(float* dst, const float* src) {
    unsigned d = (unsigned)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async16(float* dst, const float* src) {
    unsigned d = (unsigned)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
}

// grid: (column blocks, heads, requests).  Lane `sub` of a column's TPC lanes holds rows sub, sub + TPC,
// ..., R of them.  q, a, w: element (n, head, d) at [n * ld + head * dim + d] (q and w: head / heads_per_unit in
// head's place); SCALAR: a and the write
// gate b come from gates[n * gate_stride + head * 3 + {0, 1}] and column `vdim` (if cols > vdim) has the
// value 1.  v: (n, head, c) at [n * v_ld + head * vdim + c].  out: [N, heads, cols], times q_scale.
template <int R, int TPC, bool SCALAR>
__global__ void __launch_bounds__(GR_THREADS)
gated_recurrence_kernel(const float* __restrict__ q, int q_ld, const float* __restrict__ a, int a_ld,
                        const float* __restrict__ w, int w_ld, const float* __restrict__ gates,
                        int gate_stride, const float* __restrict__ v, int v_ld, float* __restrict__ state,
                        long long state_stride, const int* __restrict__ slots, const int* __restrict__ cu_q,
                        float* __restrict__ out, int heads, int heads_per_unit, int dim, int vdim, int cols,
                        float q_scale, int num_slots) {
    extern __shared__ __align__(16) float sm[];
    constexpr int COLS = GR_THREADS / TPC, DP = R * TPC;
    constexpr int ROWS = SCALAR ? 2 : 3;  // arrays of DP floats per token: q, w (, a)
    constexpr int BUF = GR_CHUNK * (ROWS * DP + COLS + 4);
    ie_pdl_trigger();
    ie_pdl_wait();
    int seq = blockIdx.z, head = blockIdx.y;
    int start = cu_q[seq], len = cu_q[seq + 1] - start;
    int slot = slots[seq];
    if (len <= 0 || slot < 0 || slot >= num_slots) return;
    const int unit = head / heads_per_unit;
    int tid = threadIdx.x;
    int sub = tid % TPC, my_col = tid / TPC, col = blockIdx.x * COLS + my_col;
    bool live = col < cols;
    float* S = state + (size_t)slot * state_stride + ((size_t)head * cols + (live ? col : 0)) * dim;
    float s[R];
#pragma unroll
    for (int i = 0; i < R; ++i) {
        int r = sub + TPC * i;
        s[i] = (live && r < dim) ? S[r] : 0.f;
    }
    // entries beyond dim (the copies never touch them) read as zero
    if (DP > dim) {
        int pad = DP - dim;
        for (int i = tid; i < GR_STAGES * GR_CHUNK * ROWS * pad; i += GR_THREADS) {
            int row = i / pad, c = dim + (i - row * pad);
            sm[(row / (GR_CHUNK * ROWS)) * BUF + (row % (GR_CHUNK * ROWS)) * DP + c] = 0.f;
        }
    }
    __syncthreads();
    int c0 = blockIdx.x * COLS;
    bool vec = (dim % 4 == 0) && (q_ld % 4 == 0) && (w_ld % 4 == 0) && (SCALAR || a_ld % 4 == 0) &&
               ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(w) |
                 (SCALAR ? 0 : reinterpret_cast<uintptr_t>(a))) % 16 == 0);
    auto stage = [&](int t0, int b) {
        int cnt = min(GR_CHUNK, len - t0);
        float* qs = sm + b * BUF;
        float* ws = qs + GR_CHUNK * DP;
        float* as = ws + GR_CHUNK * DP;  // (SCALAR: not there; vs starts here)
        float* vs = sm + b * BUF + ROWS * GR_CHUNK * DP;
        float* gs = vs + GR_CHUNK * COLS;  // a and b of the tokens (SCALAR)
        if (vec) {
            int dq = dim >> 2;
            for (int i = tid; i < cnt * dq; i += GR_THREADS) {
                int tt = i / dq, d = (i - tt * dq) * 4;
                size_t n = (size_t)(start + t0 + tt);
                cp_async16(qs + tt * DP + d, q + n * q_ld + unit * dim + d);
                cp_async16(ws + tt * DP + d, w + n * w_ld + unit * dim + d);
                if (!SCALAR) cp_async16(as + tt * DP + d, a + n * a_ld + head * dim + d);
            }
        } else {
            for (int i = tid; i < cnt * dim; i += GR_THREADS) {
                int tt = i / dim, d = i - tt * dim;
                size_t n = (size_t)(start + t0 + tt);
                cp_async4(qs + tt * DP + d, q + n * q_ld + unit * dim + d);
                cp_async4(ws + tt * DP + d, w + n * w_ld + unit * dim + d);
                if (!SCALAR) cp_async4(as + tt * DP + d, a + n * a_ld + head * dim + d);
            }
        }
        for (int i = tid; i < cnt * COLS; i += GR_THREADS) {
            int tt = i / COLS, c = i - tt * COLS;
            if (c0 + c < vdim) cp_async4(vs + tt * COLS + c, v + (size_t)(start + t0 + tt) * v_ld + head * vdim + c0 + c);
        }
        if (SCALAR && tid < 2 * cnt)
            cp_async4(gs + tid, gates + (size_t)(start + t0 + (tid >> 1)) * gate_stride + head * 3 + (tid & 1));
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    // (a step of one chunk waits for its memory once; a prompt's chunks find theirs landed: with one
    // chunk ahead every eight tokens cost a trip to memory, 0.25 us a token whatever the sizes)
    int n_chunks = (len + GR_CHUNK - 1) / GR_CHUNK;
    for (int c = 0; c < GR_STAGES - 1; ++c) {
        if (c < n_chunks) stage(c * GR_CHUNK, c);
        else asm volatile("cp.async.commit_group;" ::: "memory");
    }
    bool ones = SCALAR && live && col >= vdim;  // the normaliser's column
    for (int c = 0; c < n_chunks; ++c) {
        int t0 = c * GR_CHUNK, b = c % GR_STAGES;
        int cnt = min(GR_CHUNK, len - t0);
        asm volatile("cp.async.wait_group %0;" ::"n"(GR_STAGES - 2) : "memory");
        __syncthreads();  // this chunk has landed for everyone, and everyone is done with the buffer filled next
        if (c + GR_STAGES - 1 < n_chunks) stage((c + GR_STAGES - 1) * GR_CHUNK, (c + GR_STAGES - 1) % GR_STAGES);
        else asm volatile("cp.async.commit_group;" ::: "memory");
        const float* qs = sm + b * BUF + sub;
        const float* ws = qs + GR_CHUNK * DP;
        const float* as = ws + GR_CHUNK * DP;
        const float* vs = sm + b * BUF + ROWS * GR_CHUNK * DP + my_col;
        const float* gs = sm + b * BUF + ROWS * GR_CHUNK * DP + GR_CHUNK * COLS;
        // The chunk's tokens in order; their read-outs are summed over a column's lanes together at the
        // end, so that the exchanges of eight tokens overlap instead of each stalling the next token.
        float rds[GR_CHUNK];
#pragma unroll
        for (int tt = 0; tt < GR_CHUNK; ++tt) {
            rds[tt] = 0.f;
            if (tt < cnt) {
                float u = ones ? 1.0f : (live ? vs[tt * COLS] : 0.f);
                float a_s = 1.0f;
                if (SCALAR) { a_s = gs[2 * tt]; u *= gs[2 * tt + 1]; }
                float r4[4] = {0.f, 0.f, 0.f, 0.f};  // four partial sums: shorter chains, a fixed order
#pragma unroll
                for (int i = 0; i < R; ++i) {
                    int at = tt * DP + TPC * i;
                    float av = SCALAR ? a_s : as[at];
                    s[i] = fmaf(ws[at], u, s[i] * av);
                    r4[i & 3] = fmaf(s[i], qs[at], r4[i & 3]);
                }
                rds[tt] = (r4[0] + r4[1]) + (r4[2] + r4[3]);
            }
        }
#pragma unroll
        for (int o = TPC >> 1; o > 0; o >>= 1) {
#pragma unroll
            for (int tt = 0; tt < GR_CHUNK; ++tt) rds[tt] += __shfl_xor_sync(0xffffffffu, rds[tt], o);
        }
        if (live && sub == 0) {
#pragma unroll
            for (int tt = 0; tt < GR_CHUNK; ++tt)
                if (tt < cnt) out[((size_t)(start + t0 + tt) * heads + head) * cols + col] = rds[tt] * q_scale;
        }
    }
    if (live) {
#pragma unroll
        for (int i = 0; i < R; ++i) {
            int r = sub + TPC * i;
            if (r < dim) S[r] = s[i];
        }
    }
}

// One warp per (token, head).  o: [rows, cols]; with `gates` the column `vdim` is n . q and the
// row is first divided by max(|n . q|, exp(-m)) + 1e-6.  weight: [vdim] shared by the heads,
// [heads * vdim], or null.  gate_pre (optional): element (n, head, d) at [n * gate_ld + head * vdim + d]; the
// row is multiplied by sigmoid(gate_pre), or by silu(gate_pre) with gate_silu.
template <typename T>
__global__ void __launch_bounds__(128)
recurrence_readout_kernel(const float* __restrict__ o, int cols, const float* __restrict__ gates,
                          const float* __restrict__ weight, int weight_per_head, float eps,
                          const float* __restrict__ gate_pre, int gate_ld, int gate_silu, T* __restrict__ out,
                          long long rows, int heads, int vdim) {
    ie_pdl_trigger();
    ie_pdl_wait();
    long long row = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
    if (row >= rows) return;
    int lane = threadIdx.x & 31;
    long long n = row / heads;
    int head = (int)(row - n * heads);
    const float* src = o + row * cols;
    float den = 1.0f;
    if (gates != nullptr) den = fmaxf(fabsf(src[vdim]), gates[row * 3 + 2]) + 1e-6f;
    float ss = 0.f;
    for (int d = lane; d < vdim; d += 32) {
        float x = src[d] / den;
        ss = fmaf(x, x, ss);
    }
    ss = warp_sum(ss);
    float inv = 1.0f / sqrtf(ss / (float)vdim + eps);
    const float* wrow = weight != nullptr && weight_per_head ? weight + (size_t)head * vdim : weight;
    for (int d = lane; d < vdim; d += 32) {
        float y = (src[d] / den) * inv;
        if (weight != nullptr) y *= wrow[d];
        if (gate_pre != nullptr) {
            float gp = gate_pre[n * gate_ld + (size_t)head * vdim + d];
            y *= gate_silu ? silu_f(gp) : sigmoid_f(gp);
        }
        ie_store(out + row * vdim + d, y);
    }
}

inline int grid_for(size_t total, int threads) {
    size_t want = (total + threads - 1) / threads;
    return (int)(want < 148 * 16 ? want : 148 * 16);
}

template <int R, int TPC, bool SCALAR>
int launch_recurrence(const float* q, int q_ld, const float* a, int a_ld, const float* w, int w_ld,
                      const float* gates, int gate_stride, const float* v, int v_ld, float* state,
                      long long state_stride, const int* slots, const int* cu_q, float* out, int num_seqs, int heads,
                      int heads_per_unit, int dim, int vdim, int cols, float q_scale, int num_slots, cudaStream_t s) {
    constexpr int COLS = GR_THREADS / TPC;
    size_t smem = (size_t)GR_STAGES * GR_CHUNK * ((SCALAR ? 2 : 3) * R * TPC + COLS + 4) * sizeof(float);
    static IePerDevice allowed;
    cudaError_t e = ie_allow_smem(allowed, gated_recurrence_kernel<R, TPC, SCALAR>, 200 * 1024);  // (dim 512: 198 KB)
    if (e != cudaSuccess) return (int)e;
    dim3 grid((cols + COLS - 1) / COLS, heads, num_seqs);
    return ie_launch(gated_recurrence_kernel<R, TPC, SCALAR>, grid, dim3(GR_THREADS), smem, s, q, q_ld, a, a_ld, w,
                     w_ld, gates, gate_stride, v, v_ld, state, state_stride, slots, cu_q, out, heads, heads_per_unit, dim, vdim, cols,
                     q_scale, num_slots);
}
}  // namespace

IE_API int ie_short_conv_residual(const void* x, int dtype, const float* w, float* state, long long state_stride,
                                  const int* slots, const int* seq_of_token, const int* cu_q, void* out,
                                  int num_tokens, int num_seqs, int channels, int taps, int num_slots, int* err,
                                  void* stream) {
    if (num_tokens <= 0) return 0;
    if (taps < 1) return (int)cudaErrorInvalidValue;
    cudaStream_t s = (cudaStream_t)stream;
    int e;
    // few tokens: a thread per channel; many: a few channels per thread
    int per_row = (channels + 255) / 256;
    int cb = num_tokens >= 512 ? (per_row < 2 ? per_row : 2) : per_row;
    dim3 grid(num_tokens, cb), tail_grid(num_seqs, per_row);
    if (dtype == IE_BF16)
        e = ie_launch(short_conv_residual_kernel<__nv_bfloat16>, grid, dim3(256), 0, s,
                      (const __nv_bfloat16*)x, w, (const float*)state, state_stride, slots, seq_of_token, cu_q,
                      (__nv_bfloat16*)out, channels, taps, num_slots, err);
    else
        e = ie_launch(short_conv_residual_kernel<float>, grid, dim3(256), 0, s, (const float*)x, w,
                      (const float*)state, state_stride, slots, seq_of_token, cu_q, (float*)out, channels, taps,
                      num_slots, err);
    if (e != 0 || taps < 2) return e;
    if (dtype == IE_BF16)
        return ie_launch(short_conv_tail_kernel<__nv_bfloat16>, tail_grid, dim3(256), 0, s,
                         (const __nv_bfloat16*)x, state, state_stride, slots, cu_q, channels, taps, num_slots);
    return ie_launch(short_conv_tail_kernel<float>, tail_grid, dim3(256), 0, s, (const float*)x, state,
                     state_stride, slots, cu_q, channels, taps, num_slots);
}

IE_API int ie_rotate_heads(float* x, int ld, const int* positions, const float* table, int rot_dims,
                           int table_positions, int num_tokens, int units, int dim, int* err, void* stream) {
    if (num_tokens <= 0 || rot_dims == 0) return 0;
    if (rot_dims < 0 || rot_dims % 2 || rot_dims > dim || table == nullptr || units < 1 || (long long)units * dim > ld)
        return (int)cudaErrorInvalidValue;
    int pairs = units * (rot_dims / 2), per_row = (pairs + 127) / 128;
    // few tokens: a thread per pair; many: several pairs per thread
    dim3 grid(num_tokens, num_tokens >= 256 ? (per_row + 3) / 4 : per_row);
    return ie_launch(rotate_heads_kernel, grid, dim3(128), 0, (cudaStream_t)stream, x, ld, positions, table, rot_dims,
                     table_positions, units, dim, err);
}

IE_API int ie_lowrank_decay(const float* y, int y_ld, const float* w2, const float* bias, float inv_tau,
                            float* decay, int num_tokens, int channels, int rank, void* stream) {
    if (num_tokens <= 0 || channels <= 0) return 0;
    if (rank < 1) return (int)cudaErrorInvalidValue;
    dim3 grid((num_tokens + LD_TOKENS - 1) / LD_TOKENS, (channels + 127) / 128);
    return ie_launch(lowrank_decay_kernel, grid, dim3(128), 0, (cudaStream_t)stream, y, y_ld, w2, bias, inv_tau,
                     decay, num_tokens, channels, rank);
}

IE_API int ie_hgrn2_gates(float* proj, int ld, const float* bias, const float* lower, float* write,
                          int num_tokens, int size, void* stream) {
    size_t total = (size_t)num_tokens * size;
    if (total == 0) return 0;
    return ie_launch(hgrn2_gates_kernel, dim3(grid_for(total, 256)), dim3(256), 0, (cudaStream_t)stream, proj, ld,
                     bias, lower, write, size, total);
}

IE_API int ie_mlstm_gates(const float* gi, const float* gf, int ld, const float* bias_i, const float* bias_f,
                          float cap, float* state, long long state_stride, long long m_offset, const int* slots,
                          const int* cu_q, float* gates, int num_seqs, int heads, int num_slots, void* stream) {
    if (num_seqs <= 0 || heads <= 0) return 0;
    return ie_launch(mlstm_gates_kernel, dim3(heads, num_seqs), dim3(32), 0, (cudaStream_t)stream, gi, gf, ld,
                     bias_i, bias_f, cap, state, state_stride, m_offset, slots, cu_q, gates, heads, num_slots);
}

// gates == nullptr: a and w per head and channel (a, a_ld given); else the gates' scalars, a token's
// `gate_stride` numbers apart (0: the same for every token).
IE_API int ie_gated_recurrence(const float* q, int q_ld, const float* a, int a_ld, const float* w, int w_ld,
                               const float* gates, int gate_stride, const float* v, int v_ld, float* state,
                               long long state_stride, const int* slots, const int* cu_q, float* out, int num_seqs, int heads,
                               int heads_per_unit, int dim, int vdim, int cols, float q_scale, int num_slots, void* stream) {
    if (num_seqs <= 0) return 0;
    if (heads_per_unit < 1 || heads % heads_per_unit) return (int)cudaErrorInvalidValue;
    if (cols < vdim || cols > vdim + 1 || (gates == nullptr && (a == nullptr || cols != vdim)))
        return (int)cudaErrorInvalidValue;
    cudaStream_t s = (cudaStream_t)stream;
#define IE_GR_ARGS q, q_ld, a, a_ld, w, w_ld, gates, gate_stride, v, v_ld, state, state_stride, slots, cu_q, out, num_seqs, heads, heads_per_unit, dim, vdim, cols, q_scale, num_slots, s
#define IE_GR_PICK(SC)                                                        \
    if (dim <= 8) return launch_recurrence<8, 1, SC>(IE_GR_ARGS);             \
    if (dim <= 16) return launch_recurrence<8, 2, SC>(IE_GR_ARGS);            \
    if (dim <= 32) return launch_recurrence<8, 4, SC>(IE_GR_ARGS);            \
    if (dim <= 64) return launch_recurrence<8, 8, SC>(IE_GR_ARGS);            \
    if (dim <= 128) return launch_recurrence<8, 16, SC>(IE_GR_ARGS);          \
    if (dim <= 256) return launch_recurrence<8, 32, SC>(IE_GR_ARGS);          \
    if (dim <= 512) return launch_recurrence<16, 32, SC>(IE_GR_ARGS);
    if (gates != nullptr) { IE_GR_PICK(true) } else { IE_GR_PICK(false) }
#undef IE_GR_PICK
#undef IE_GR_ARGS
    return (int)cudaErrorInvalidValue;  // dim <= 512
}

IE_API int ie_recurrence_readout(const float* o, int cols, const float* gates, const float* weight,
                                 int weight_per_head, float eps, const float* gate_pre, int gate_ld, int gate_silu,
                                 void* out, int out_dtype, long long rows, int heads, int vdim, void* stream) {
    if (rows <= 0) return 0;
    dim3 grid((unsigned)((rows + 3) / 4));
    cudaStream_t s = (cudaStream_t)stream;
    if (out_dtype == IE_BF16)
        return ie_launch(recurrence_readout_kernel<__nv_bfloat16>, grid, dim3(128), 0, s, o, cols, gates, weight,
                         weight_per_head, eps, gate_pre, gate_ld, gate_silu, (__nv_bfloat16*)out, rows, heads, vdim);
    return ie_launch(recurrence_readout_kernel<float>, grid, dim3(128), 0, s, o, cols, gates, weight,
                     weight_per_head, eps, gate_pre, gate_ld, gate_silu, (float*)out, rows, heads, vdim);
}

// `out_dtype`: of the convolved values.  gates == nullptr: the convolution alone.
IE_API int ie_conv_silu(const float* x, int x_ld, const float* w, const float* bias, const float* state,
                        long long state_stride, long long tail_at, const int* slots, const int* seq_of_token,
                        const int* cu_q, void* out, int out_ld, int out_dtype, int num_tokens, int channels, int taps,
                        int num_slots, const float* dt_pre, const float* dt_bias, const float* A_log, float* gates,
                        int heads, int* err, void* stream) {
    if (num_tokens <= 0) return 0;
    if (taps < 1 || channels < 1 || out_ld < channels) return (int)cudaErrorInvalidValue;
    cudaStream_t s = (cudaStream_t)stream;
    dim3 grid((num_tokens + CS_TOKENS - 1) / CS_TOKENS, (channels + 127) / 128 + 1);
    if (gates == nullptr) heads = 0;
#define IE_CS_LAUNCH(T, TAPS)                                                                                        \
    return ie_launch(conv_silu_kernel<T, TAPS>, grid, dim3(128), 0, s, x, x_ld, w, bias, state, state_stride,        \
                     tail_at, slots, seq_of_token, cu_q, (T*)out, out_ld, num_tokens, channels, taps, num_slots,     \
                     dt_pre, dt_bias, A_log, gates, heads, err)
#define IE_CS_PICK(T)                      \
    if (taps == 2) IE_CS_LAUNCH(T, 2);     \
    if (taps == 3) IE_CS_LAUNCH(T, 3);     \
    if (taps == 4) IE_CS_LAUNCH(T, 4);     \
    IE_CS_LAUNCH(T, 0)
    if (out_dtype == IE_BF16) { IE_CS_PICK(__nv_bfloat16); }
    IE_CS_PICK(float);
#undef IE_CS_PICK
#undef IE_CS_LAUNCH
}

// x, z, raw may be null: no skip, no gate, no kept inputs to move on.
IE_API int ie_gated_group_norm(const float* y, const float* x, int x_ld, const float* skip, const float* z, int z_ld,
                               const float* weight, float eps, void* out, int out_ld, int out_dtype, int num_tokens,
                               int size, int parts, int vdim, const float* raw, int raw_ld, float* state,
                               long long state_stride, long long tail_at, const int* slots, const int* cu_q, int num_seqs,
                               int channels, int taps, int num_slots, void* stream) {
    if (num_tokens <= 0) return 0;
    if (parts < 1 || size % parts || vdim < 1 || out_ld < size) return (int)cudaErrorInvalidValue;
    size_t smem = (size_t)(size / parts) * sizeof(float);
    if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
    cudaStream_t s = (cudaStream_t)stream;
    const int width = size / parts, mine = raw != nullptr && taps > 1 ? num_seqs * ((channels + GN_THREADS - 1) / GN_THREADS) : 0;
    const bool vec = x == nullptr && z == nullptr && width % 4 == 0 && width <= GN_THREADS * 16 && out_ld % 4 == 0 &&
                     ((reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(weight)) % 16 == 0) &&
                     reinterpret_cast<uintptr_t>(out) % (out_dtype == IE_BF16 ? 8 : 16) == 0;
#define IE_GG_LAUNCH(T, V)                                                                                           \
    do {                                                                                                             \
        static IePerDevice allowed;                                                                                  \
        if (!V && smem > 40 * 1024) {                                                                                \
            cudaError_t e = ie_allow_smem(allowed, gated_group_norm_kernel<T, V>, 200 * 1024);                       \
            if (e != cudaSuccess) return (int)e;                                                                     \
        }                                                                                                            \
        return ie_launch(gated_group_norm_kernel<T, V>, dim3((unsigned)(num_tokens * parts + mine)),                 \
                         dim3(GN_THREADS), V ? 0 : smem, s, y, x, x_ld, skip, z, z_ld, weight, eps, (T*)out, out_ld, \
                         num_tokens, size, parts, vdim, raw, raw_ld, state, state_stride, tail_at, slots, cu_q,      \
                         channels, taps, num_slots);                                                                 \
    } while (0)
    if (out_dtype == IE_BF16) {
        if (vec) IE_GG_LAUNCH(__nv_bfloat16, true);
        IE_GG_LAUNCH(__nv_bfloat16, false);
    }
    if (vec) IE_GG_LAUNCH(float, true);
    IE_GG_LAUNCH(float, false);
#undef IE_GG_LAUNCH
}
