// Attention over shared latent rows on the tensor cores (bfloat16).  Built per (key row size LM_DK, value row size
// LM_DV), both multiples of 8, LM_DV <= LM_DK and at most 512.
//
// Every query head of a token attends over the same cached rows: a key is a whole row (LM_DK
// entries: the latent, then the rotated part), its value the row's first LM_DV entries.  So the rows
// of the score matrix are (token, head) pairs of one request, and a block streams the request's
// rows once for all of its pairs: 16 pairs and 64-key tiles where requests bring a token or two
// (decoding), 64 pairs and 32-key tiles where they bring portions of prompts (a key tile then
// serves four times the rows).  Eight warps:
//   scores   a warp takes eight keys of the tile (and a share of the rows' 16-row tiles):
//            S = Q K^T over LM_DK by mma.sync.m16n8k16, Q and the key tile in shared memory (key tiles
//            arrive by cp.async, two buffers);
//   softmax  a few threads per row: mask (a row sees positions up to its own), running maximum
//            and sum in 32-bit, a weight as two bfloat16 terms (its rounded value and the remainder: 16 bits
//            of its mantissa) into shared memory; a sink (`sinks`, a number per head) is one more term
//            of the sum that has no key and no value: a row starts from it, or the merge adds it;
//   values   warp w owns every eighth 8-column slice of the LM_DV output columns: O = O * alpha + P V,
//            V's fragments straight from the key tile with ldmatrix.trans.
// A context may be cut into `splits` ranges of key tiles (few requests, long contexts): the blocks of
// a range leave maximum, sum and the unnormalised output in scratch, and a second kernel adds the
// ranges in order.  Rows, sums and the order of additions depend on the request alone.
#include "common.cuh"
#include <math.h>

#ifndef LM_DK
#define LM_DK 576
#endif
#ifndef LM_DV
#define LM_DV 512
#endif

namespace {

constexpr int DK = LM_DK, DV = LM_DV;
static_assert(DK % 8 == 0 && DV % 8 == 0 && DV <= DK && DV <= 512, "sizes");
constexpr int DKP = (DK + 15) / 16 * 16;  // columns beyond DK read as zero in both operands
constexpr int LD = DKP + 8;               // rows 16 bytes longer: ldmatrix rows fall on different banks
constexpr int CHUNKS = DK / 8;            // 16-byte pieces of a row
constexpr float LM_LOG2E = 1.4426950408889634f;  // scores, maxima and the parts' maxima are in units of log2 e

__device__ __forceinline__ void cp_async16(void* dst, const void* src, int src_bytes) {
    unsigned d = (unsigned)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(src_bytes) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ void mma_bf16(float* c, const unsigned* a, const unsigned* b) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}

struct LmSmem {
    __nv_bfloat16* q;   // [rows][ld]
    __nv_bfloat16* k;   // [BUFS][keys][ld]
    float* s;           // [rows][keys + 4]
    __nv_bfloat16* p;   // [2][rows][keys + 8]: the weights rounded, and what the rounding left
    float* alpha;       // [rows]
    float* m;           // [rows]
    float* l;           // [rows]
};

constexpr size_t lm_smem_bytes(int rows, int keys, int bufs) {
    return (size_t)(rows + bufs * keys) * LD * 2 + rows * (keys + 4) * 4 + 2 * rows * (keys + 8) * 2 + 3 * rows * 4;
}

// grid: (row tiles of a request, requests, splits).  MT 16-row tiles and KEYS keys per step, LM_WARPS warps.  With
// BUFS 2 a tile's three phases follow one another; with BUFS 3 (a third key tile in shared memory) the scores of
// the next tile and the values of this one are one phase, so a tile costs two barriers instead of three and the
// two products, which do not depend on each other, overlap.
template <int MT, int KEYS, int LM_WARPS, int BUFS>
__global__ void __launch_bounds__(LM_WARPS * 32)
latent_attention_mma_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ cache,
                            const int* __restrict__ block_tables, int table_width, const int* __restrict__ cu_q,
                            const int* __restrict__ ctx_lens, __nv_bfloat16* __restrict__ out,
                            float* __restrict__ scratch, int heads, int page_size,
                            int total_pages, float scale, const float* __restrict__ sinks, int splits, int* err) {
    extern __shared__ __align__(16) unsigned char raw[];
    constexpr int LM_ROWS = 16 * MT, LM_KEYS = KEYS, LM_THREADS = LM_WARPS * 32;
    constexpr int SLICES = DV / 8, PER_WARP = (SLICES + LM_WARPS - 1) / LM_WARPS;  // 8-column slices of the output; of a warp
    constexpr int KEYS_PER_WARP = KEYS / LM_WARPS;  // keys a warp brings
    constexpr int N_TILES = KEYS / 8;            // 8-key slices of a key tile
    constexpr int WPM = LM_WARPS / MT;           // warps that share sixteen rows, each with NPW slices of keys
    constexpr int NPW = N_TILES / WPM;
    constexpr int TPR = LM_THREADS / LM_ROWS;    // softmax threads per row
    constexpr int KPT = KEYS / TPR;              // ... and keys per thread
    static_assert(LM_WARPS % MT == 0 && N_TILES % WPM == 0 && (NPW == 1 || NPW == 2) && KPT % 4 == 0 && TPR <= 32, "shape");
    ie_pdl_trigger();
    ie_pdl_wait();
    // (the blocks of a request's last rows see the most keys: they start first)
    int seq = blockIdx.y, tile = gridDim.x - 1 - blockIdx.x, split = blockIdx.z;
    int q0 = cu_q[seq], q_len = cu_q[seq + 1] - q0;
    int rows_total = q_len * heads;
    int row0 = tile * LM_ROWS;
    if (row0 >= rows_total) return;
    int ctx_len = ctx_lens[seq];
    int start = ctx_len - q_len;  // position of the request's first token of this step
    int rows_here = min(LM_ROWS, rows_total - row0);
    int last_pos = start + (row0 + rows_here - 1) / heads;  // the last position any row of the block sees
    int tiles_all = last_pos / LM_KEYS + 1;
    int per = (tiles_all + splits - 1) / splits;
    int t_begin = split * per, t_end = min(tiles_all, t_begin + per);

    LmSmem sm;
    sm.q = reinterpret_cast<__nv_bfloat16*>(raw);
    sm.k = sm.q + LM_ROWS * LD;
    sm.s = reinterpret_cast<float*>(sm.k + BUFS * LM_KEYS * LD);
    sm.p = reinterpret_cast<__nv_bfloat16*>(sm.s + LM_ROWS * (LM_KEYS + 4));
    sm.alpha = reinterpret_cast<float*>(sm.p + 2 * LM_ROWS * (LM_KEYS + 8));
    sm.m = sm.alpha + LM_ROWS;
    sm.l = sm.m + LM_ROWS;

    int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
    const int* table = block_tables + (size_t)seq * table_width;
    int page_shift = 31 - __clz(page_size);  // (pages hold a power of two of tokens)

    if (DKP > DK) {
        for (int i = tid; i < (LM_ROWS + BUFS * LM_KEYS) * (DKP - DK); i += LM_THREADS) {
            int r = i / (DKP - DK > 0 ? DKP - DK : 1), c = DK + i % (DKP - DK > 0 ? DKP - DK : 1);
            sm.q[r * LD + c] = __float2bfloat16_rn(0.f);  // (q and k are one array of rows)
        }
    }
    auto load_keys = [&](int t, int buf) {
        // a warp takes whole keys, its lanes their pieces; the looks into the block table first, all at once
        __nv_bfloat16* dst = sm.k + ((size_t)buf * LM_KEYS + warp * KEYS_PER_WARP) * LD;
        int pages[KEYS_PER_WARP];
        const int pos0 = t * LM_KEYS + warp * KEYS_PER_WARP;
#pragma unroll
        for (int j = 0; j < KEYS_PER_WARP; ++j) pages[j] = pos0 + j <= last_pos ? table[(pos0 + j) >> page_shift] : 0;
#pragma unroll
        for (int j = 0; j < KEYS_PER_WARP; ++j) {
            const int pos = pos0 + j, page = pages[j];
            bool there = pos <= last_pos;
            if (there && (page < 0 || page >= total_pages)) {
                ie_report(err, page < 0 ? IE_ERR_TABLE : IE_ERR_PAGE, page, seq);
                there = false;
            }
            const __nv_bfloat16* src = there ? cache + ((size_t)page * page_size + (pos & (page_size - 1))) * DK : cache;
#pragma unroll
            for (int c0 = 0; c0 < CHUNKS; c0 += 32) {
                int c = c0 + lane;
                if (c < CHUNKS) cp_async16(dst + j * LD + c * 8, src + c * 8, there ? 16 : 0);
            }
        }
        cp_async_commit();
    };
    if (t_begin < t_end) load_keys(t_begin, 0);
    // queries: row r of the block is (token (row0 + r) / heads, head (row0 + r) % heads)
    for (int i = tid; i < LM_ROWS * CHUNKS; i += LM_THREADS) {
        int r = i / CHUNKS, c = i - r * CHUNKS;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (r < rows_here) {
            int rr = row0 + r;
            v = *reinterpret_cast<const uint4*>(q + ((size_t)(q0 + rr / heads) * heads + rr % heads) * DK + c * 8);
        }
        *reinterpret_cast<uint4*>(sm.q + r * LD + c * 8) = v;
    }
    if (tid < LM_ROWS) {  // (cut contexts: the merge adds the sink's term)
        bool with_sink = sinks != nullptr && splits == 1 && tid < rows_here;
        sm.m[tid] = with_sink ? sinks[(row0 + tid) % heads] * LM_LOG2E : -INFINITY;
        sm.l[tid] = with_sink ? 1.f : 0.f;
    }

    float acc[MT][PER_WARP][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int i = 0; i < PER_WARP; ++i) acc[mt][i][0] = acc[mt][i][1] = acc[mt][i][2] = acc[mt][i][3] = 0.f;
    // (warp w owns slices w, w + LM_WARPS, ...)

    // scores: this warp's keys (eight, or sixteen with NPW 2) against its sixteen rows, even and odd steps of
    // k in sums of their own
    auto scores = [&](const __nv_bfloat16* ks) {
        const int ns = (warp % WPM) * NPW, m_tile = warp / WPM;
        float c[NPW][2][4];
#pragma unroll
        for (int i = 0; i < NPW; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) c[i][0][e] = c[i][1][e] = 0.f;
        // fragments by ldmatrix: A (16 x 16 of Q) one x4; B one x4: 8 keys x 32 of k, or 16 keys x 16
        unsigned qa = (unsigned)__cvta_generic_to_shared(sm.q + (m_tile * 16 + (lane & 15)) * LD + (lane >> 4) * 8);
        const int brow = NPW == 1 ? (lane & 7) : (lane & 7) + ((lane >> 4) << 3), bcol = NPW == 1 ? (lane >> 3) * 8 : ((lane >> 3) & 1) * 8;
        unsigned kb = (unsigned)__cvta_generic_to_shared(ks + (ns * 8 + brow) * LD + bcol);
        int kk = 0;
#pragma unroll 6
        for (; kk + 32 <= DKP; kk += 32) {
            unsigned a[2][4], b[NPW][4];
#pragma unroll
            for (int h = 0; h < 2; ++h)
                asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                             : "=r"(a[h][0]), "=r"(a[h][1]), "=r"(a[h][2]), "=r"(a[h][3]) : "r"(qa + (kk + h * 16) * 2));
#pragma unroll
            for (int i = 0; i < NPW; ++i)
                asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                             : "=r"(b[i][0]), "=r"(b[i][1]), "=r"(b[i][2]), "=r"(b[i][3]) : "r"(kb + (kk + i * 16) * 2));
#pragma unroll
            for (int h = 0; h < 2; ++h)
#pragma unroll
                for (int i = 0; i < NPW; ++i) mma_bf16(c[i][h], a[h], NPW == 1 ? b[0] + 2 * h : b[h % NPW] + 2 * i);
        }
        if (kk < DKP) {  // a last step of 16
            unsigned a[4], b[4];
            asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                         : "=r"(a[0]), "=r"(a[1]), "=r"(a[2]), "=r"(a[3]) : "r"(qa + kk * 2));
            if (NPW == 1) {
                unsigned kb2 = (unsigned)__cvta_generic_to_shared(ks + (ns * 8 + (lane & 7)) * LD + ((lane >> 3) & 1) * 8);
                asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(b[0]), "=r"(b[1]) : "r"(kb2 + kk * 2));
            } else {
                asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                             : "=r"(b[0]), "=r"(b[1]), "=r"(b[2]), "=r"(b[3]) : "r"(kb + kk * 2));
            }
#pragma unroll
            for (int i = 0; i < NPW; ++i) mma_bf16(c[i][0], a, b + 2 * i);
        }
        const float sl2 = scale * LM_LOG2E;
#pragma unroll
        for (int i = 0; i < NPW; ++i) {
            float* s0 = sm.s + (m_tile * 16 + g) * (LM_KEYS + 4) + (ns + i) * 8 + 2 * t4;
            *reinterpret_cast<float2*>(s0) = make_float2((c[i][0][0] + c[i][1][0]) * sl2, (c[i][0][1] + c[i][1][1]) * sl2);
            *reinterpret_cast<float2*>(s0 + 8 * (LM_KEYS + 4)) = make_float2((c[i][0][2] + c[i][1][2]) * sl2, (c[i][0][3] + c[i][1][3]) * sl2);
        }
    };
    // softmax: TPR threads per row, KPT keys each
    auto softmax = [&](int t) {
        int r = tid / TPR, j = tid % TPR;
        int rr = row0 + r;
        int pos_r = r < rows_here ? start + rr / heads : -1;
        float v[KPT], mx = -INFINITY;
#pragma unroll
        for (int i = 0; i < KPT; ++i) {
            int kp = t * LM_KEYS + j * KPT + i;
            v[i] = kp <= pos_r ? sm.s[r * (LM_KEYS + 4) + j * KPT + i] : -INFINITY;
            mx = fmaxf(mx, v[i]);
        }
#pragma unroll
        for (int o = TPR / 2; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        float m_old = sm.m[r];
        float m_new = fmaxf(m_old, mx);
        float sum = 0.f;
        __align__(8) __nv_bfloat16 pb[KPT];
        __align__(8) __nv_bfloat16 pr[KPT];
#pragma unroll
        for (int i = 0; i < KPT; ++i) {
            float pv = (v[i] == -INFINITY) ? 0.f : exp2f(v[i] - m_new);
            pb[i] = __float2bfloat16_rn(pv);
            pr[i] = __float2bfloat16_rn(pv - __bfloat162float(pb[i]));
            sum += pv;
        }
#pragma unroll
        for (int o = TPR / 2; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
#pragma unroll
        for (int i = 0; i < KPT; i += 4) {
            *reinterpret_cast<uint2*>(sm.p + r * (LM_KEYS + 8) + j * KPT + i) = *reinterpret_cast<uint2*>(pb + i);
            *reinterpret_cast<uint2*>(sm.p + (LM_ROWS + r) * (LM_KEYS + 8) + j * KPT + i) = *reinterpret_cast<uint2*>(pr + i);
        }
        if (j == 0) {
            float a = (m_old == -INFINITY) ? 0.f : exp2f(m_old - m_new);
            if (m_new == -INFINITY) a = 1.f;
            sm.alpha[r] = a;
            sm.m[r] = m_new;
            sm.l[r] = sm.l[r] * a + sum;
        }
    };
    // values
    auto values = [&](const __nv_bfloat16* ks) {
        unsigned pa[MT][LM_KEYS / 16][4], pl[MT][LM_KEYS / 16][4];
        float a0[MT], a1[MT];
        bool moved = false;
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
            a0[mt] = sm.alpha[mt * 16 + g];
            a1[mt] = sm.alpha[mt * 16 + g + 8];
            moved = moved || a0[mt] != 1.f || a1[mt] != 1.f;
            unsigned pr = (unsigned)__cvta_generic_to_shared(sm.p + (mt * 16 + (lane & 15)) * (LM_KEYS + 8) + (lane >> 4) * 8);
#pragma unroll
            for (int kk = 0; kk < LM_KEYS / 16; ++kk)
                asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                             : "=r"(pa[mt][kk][0]), "=r"(pa[mt][kk][1]), "=r"(pa[mt][kk][2]), "=r"(pa[mt][kk][3])
                             : "r"(pr + kk * 32));
#pragma unroll
            for (int kk = 0; kk < LM_KEYS / 16; ++kk)
                asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                             : "=r"(pl[mt][kk][0]), "=r"(pl[mt][kk][1]), "=r"(pl[mt][kk][2]), "=r"(pl[mt][kk][3])
                             : "r"(pr + LM_ROWS * (LM_KEYS + 8) * 2 + kk * 32));
        }
        moved = __any_sync(0xffffffffu, moved);  // (mostly false once the rows' maxima have settled)
#pragma unroll
        for (int i = 0; i < PER_WARP; ++i) {
            int nt = warp + i * LM_WARPS;
            if (nt >= SLICES) break;
#pragma unroll
            for (int mt = 0; mt < MT; ++mt) {
                if (moved) { acc[mt][i][0] *= a0[mt]; acc[mt][i][1] *= a0[mt]; acc[mt][i][2] *= a1[mt]; acc[mt][i][3] *= a1[mt]; }
            }
            unsigned b[LM_KEYS / 16][2];
#pragma unroll
            for (int kk = 0; kk < LM_KEYS / 16; kk += 2) {  // 32 keys of eight columns
                unsigned addr = (unsigned)__cvta_generic_to_shared(ks + (kk * 16 + lane) * LD + nt * 8);
                asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                             : "=r"(b[kk][0]), "=r"(b[kk][1]), "=r"(b[kk + 1][0]), "=r"(b[kk + 1][1]) : "r"(addr));
            }
#pragma unroll
            for (int kk = 0; kk < LM_KEYS / 16; ++kk)
#pragma unroll
                for (int mt = 0; mt < MT; ++mt) {
                    mma_bf16(acc[mt][i], pa[mt][kk], b[kk]);
                    mma_bf16(acc[mt][i], pl[mt][kk], b[kk]);
                }
        }
    };
    auto key_tile = [&](int buf) { return sm.k + (size_t)buf * LM_KEYS * LD; };
    if constexpr (BUFS == 3) {
        if (t_begin < t_end) {
            if (t_begin + 1 < t_end) load_keys(t_begin + 1, 1);
            else cp_async_commit();
            cp_async_wait<1>();
            __syncthreads();
            scores(key_tile(0));
            __syncthreads();
        }
        for (int t = t_begin; t < t_end; ++t) {
            const int at = (t - t_begin) % 3, next = at == 2 ? 0 : at + 1;
            softmax(t);
            cp_async_wait<0>();
            __syncthreads();  // the weights are there, and so is the next tile; everyone is done with the tile before
            if (t + 2 < t_end) load_keys(t + 2, next == 2 ? 0 : next + 1);
            if (t + 1 < t_end) scores(key_tile(next));
            values(key_tile(at));
            __syncthreads();
        }
    } else {
        for (int t = t_begin; t < t_end; ++t) {
            int buf = (t - t_begin) & 1;
            cp_async_wait<0>();
            __syncthreads();
            if (t + 1 < t_end) load_keys(t + 1, buf ^ 1);
            scores(key_tile(buf));
            __syncthreads();
            softmax(t);
            __syncthreads();
            values(key_tile(buf));
        }
    }
    cp_async_wait<0>();
    __syncthreads();
    // write: normalised if the block saw the whole context, else the parts for the second kernel
#pragma unroll
    for (int i = 0; i < PER_WARP; ++i) {
        int nt = warp + i * LM_WARPS;
        if (nt >= SLICES) break;
#pragma unroll
        for (int mh = 0; mh < 2 * MT; ++mh) {
            int mt = mh >> 1, half = mh & 1;
            int r = mt * 16 + g + half * 8;
            if (r >= rows_here) continue;
            int rr = row0 + r;
            int col = nt * 8 + 2 * t4;
            float v0 = acc[mt][i][half * 2], v1 = acc[mt][i][half * 2 + 1];
            if (splits == 1) {
                float inv = sm.l[r] > 0.f ? 1.0f / sm.l[r] : 0.f;
                __nv_bfloat16* dst = out + ((size_t)(q0 + rr / heads) * heads + rr % heads) * DV + col;
                *reinterpret_cast<__nv_bfloat162*>(dst) = __floats2bfloat162_rn(v0 * inv, v1 * inv);
            } else {
                float* dst = scratch + (((size_t)(q0 * heads + rr)) * splits + split) * (DV + 2) + 2 + col;
                *reinterpret_cast<float2*>(dst) = make_float2(v0, v1);
            }
        }
    }
    if (splits > 1 && tid < rows_here) {
        float* dst = scratch + (((size_t)(q0 * heads + row0 + tid)) * splits + split) * (DV + 2);
        dst[0] = sm.m[tid];
        dst[1] = sm.l[tid];
    }
}

constexpr int LM_MAX_SPLITS = 32;
// One block per (token, head) row: the ranges' parts added in order.
__global__ void __launch_bounds__(128)
latent_attention_merge_kernel(const float* __restrict__ scratch, __nv_bfloat16* __restrict__ out, int splits,
                              const float* __restrict__ sinks, int heads) {
    ie_pdl_trigger();
    ie_pdl_wait();
    size_t row = blockIdx.x;
    const float* base = scratch + row * splits * (DV + 2);
    // the ranges' maxima and sums first, all at once (a range per thread), then the rows
    __shared__ float s_m[LM_MAX_SPLITS], s_l[LM_MAX_SPLITS];
    if ((int)threadIdx.x < splits) {
        s_m[threadIdx.x] = base[(size_t)threadIdx.x * (DV + 2)];
        s_l[threadIdx.x] = base[(size_t)threadIdx.x * (DV + 2) + 1];
    }
    const float sink = sinks != nullptr ? sinks[row % heads] * LM_LOG2E : -INFINITY;
    __syncthreads();
    float m = sink;
    for (int s = 0; s < splits; ++s) m = fmaxf(m, s_m[s]);
    float l = sinks != nullptr ? exp2f(sink - m) : 0.f;
    constexpr int PER = (DV + 127) / 128;
    float o[PER];
#pragma unroll
    for (int i = 0; i < PER; ++i) o[i] = 0.f;
#pragma unroll 4
    for (int s = 0; s < splits; ++s) {
        const float* part = base + (size_t)s * (DV + 2) + 2;
        const bool empty = s_m[s] == -INFINITY;  // (an empty range: its sums count for nothing)
        const float w = empty ? 0.f : exp2f(s_m[s] - m);
        l = fmaf(s_l[s], w, l);
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            int c = i * 128 + threadIdx.x;
            float v = c < DV && !empty ? part[c] : 0.f;
            o[i] = fmaf(v, w, o[i]);
        }
    }
    float inv = l > 0.f ? 1.0f / l : 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        int c = i * 128 + threadIdx.x;
        if (c < DV) out[row * DV + c] = __float2bfloat16_rn(o[i] * inv);
    }
}

constexpr int BUFS64 = lm_smem_bytes(64, 32, 3) <= 220 * 1024 ? 3 : 2;
IePerDevice g_lm_smem, g_lm_smem64;
}  // namespace

IE_API int ie_latent_attention_dims(int* dk, int* dv) {
    *dk = DK;
    *dv = DV;
    return lm_smem_bytes(16, 64, 2) <= 220 * 1024 && lm_smem_bytes(64, 32, 2) <= 220 * 1024;
}

// Rows (token, head pairs) a block takes: 64 when the step's longest request brings at least that
// many (portions of prompts), else 16.
IE_API int ie_latent_attention_rows(int longest_rows) { return longest_rows >= 64 ? 64 : 16; }

// scratch floats for `splits` > 1: tokens * heads * splits * (dv + 2)
IE_API int ie_latent_attention_mma(const void* q, const void* cache, const int* block_tables, int table_width,
                                   const int* cu_q, const int* ctx_lens, void* out, float* scratch, int num_tokens,
                                   int num_seqs, int max_tiles, int rows, int heads, int page_size,
                                   int total_pages, float scale, const float* sinks, int splits, int* err, void* stream) {
    if (num_seqs <= 0 || max_tiles <= 0) return 0;
    if (page_size < 1 || (page_size & (page_size - 1)) || splits < 1 || splits > LM_MAX_SPLITS || (splits > 1 && scratch == nullptr)) return (int)cudaErrorInvalidValue;
    if (rows != 16 && rows != 64) return (int)cudaErrorInvalidValue;
    cudaStream_t s = (cudaStream_t)stream;
    int rc;
#define IE_LM_ARGS (const __nv_bfloat16*)q, (const __nv_bfloat16*)cache, block_tables, table_width, cu_q, ctx_lens, \
                   (__nv_bfloat16*)out, scratch, heads, page_size, total_pages, scale, sinks, splits, err
    if (rows == 64) {
        // (sixteen warps instead of eight take as long: 636 against 633 us on 2,048 tokens of 16 heads)
        cudaError_t e = ie_allow_smem(g_lm_smem64, latent_attention_mma_kernel<4, 32, 8, BUFS64>, 220 * 1024);
        if (e != cudaSuccess) return (int)e;
        rc = ie_launch(latent_attention_mma_kernel<4, 32, 8, BUFS64>, dim3(max_tiles, num_seqs, splits), dim3(8 * 32),
                       lm_smem_bytes(64, 32, BUFS64), s, IE_LM_ARGS);
    } else {
        cudaError_t e = ie_allow_smem(g_lm_smem, latent_attention_mma_kernel<1, 64, 8, 2>, 220 * 1024);
        if (e != cudaSuccess) return (int)e;
        rc = ie_launch(latent_attention_mma_kernel<1, 64, 8, 2>, dim3(max_tiles, num_seqs, splits), dim3(8 * 32),
                       lm_smem_bytes(16, 64, 2), s, IE_LM_ARGS);
    }
#undef IE_LM_ARGS
    if (rc != 0 || splits == 1) return rc;
    return ie_launch(latent_attention_merge_kernel, dim3(num_tokens * heads), dim3(128), 0, s, (const float*)scratch,
                     (__nv_bfloat16*)out, splits, sinks, heads);
}
