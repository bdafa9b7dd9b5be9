// A linear recurrence with ONE DECAY PER KEY CHANNEL: the state is a matrix S [N, V] per head and
// request, carried in 32-bit from token to token,
//
//     S  <-  diag(a) S + k v^T            (a = exp(log_a), log_a <= 0, one per head and key channel)
//
// and the read-out is one of two:
//     o = scale * S^T q                   (u null: it sees the new state; gated linear attention)
//     o = scale * (S_old + diag(u) k v^T)^T q      (the old state, and the token's own write weighted
//                                         by u [H, N]; time mixing with a bonus)
//
// The state is stored [slots, H, V, N]; log_a is float [tokens, H N].
//
// channel_scan_kernel (any sizes): columns of S are independent.  LPC lanes share a column (EPL
// elements each, in quads), a CTA of 8 warps takes 8 * 32 / LPC columns of one (row, head) and walks
// the row's tokens in order, some of them staged in shared memory at a time.  It serves decoding (one
// token) and short portions.
//
// Long portions run in chunks of TC = 64 tokens, in both dtypes.  With L_t the channels' sums of log_a
// up to token t of a chunk, E_t = L_t (or, with the bonus, L_(t-1): what the read-out sees has not
// decayed by the token itself) and S0 the state at the chunk's start,
//
//     weights   A_ts = sum_n q_t[n] k_s[n] e^{E_t[n] - L_s[n]}  for s < t,  A_tt = q_t . k_t (bonus:
//               sum_n q_t[n] u[n] k_t[n])
//     state     dS   = sum_s (e^{L_last - L_s} * k_s) v_s^T                (every chunk at once)
//     pass      S0 of the next chunk = diag(e^{L_last}) S0 + dS            (elementwise)
//     out       o_t  = S0^T (e^{E_t} * q_t) + sum_{s <= t} A_ts v_s
//
// Every exponent is at most 0, however strong the decays: inside blocks of BT = 16 tokens the weights
// are formed pair by pair and channel by channel; between blocks the exponent is split at the blocks'
// borders, e^{E_t - start of t's block} * e^{blocks between} * e^{end of s's block - L_s}, whose factors
// go to q and k beforehand.  In 32-bit, and for the weights in both dtypes, these are fused
// multiply-adds on the CUDA cores.  The other products of bfloat16 rows run on the tensor cores
// (mma.sync from shared memory: the contractions are small and need no TMEM accumulator's set-up):
// what is 32-bit in them (decayed keys and queries, the state, the weights) goes in as three bfloat16
// parts that hold all of its 24 bits, and where both operands are 32-bit the six products of parts
// that reach above 2^-24 are formed, all accumulated in 32-bit.
#include "scan_chunks.cuh"

namespace sllm {

constexpr int BT = 16;              // tokens of a block inside a chunk
constexpr int NB = TC / BT;

struct ChannelArgs {
    const void* q; int64_t ldq;          // [tokens, >= H * N]
    const void* k; int64_t ldk;          // [tokens, >= H * N]
    const void* v; int64_t ldv;          // [tokens, >= H * V]
    const float* log_a;                  // [tokens, H * N]
    const float* u;                      // [H * N] or null
    float* state;                        // [slots, H, V, N]
    const int* row_start; const int* row_slot;
    float* out;                          // [tokens, H * V]
    float scale;
    int H, N, V;
    int vec4;                            // rows of q, k and log_a allow reads of four elements
    int vec8;                            // rows of v allow reads of eight elements
    int min_chunked;                     // rows of at least so many tokens are the chunk kernels'
    int n_rows;
    // chunk kernels only
    float* dS;                           // [slots of chunks, H, V, N]
    float* decay;                        // [slots of chunks, H, N]: L of the chunk's last token
    float* weights;                      // [slots of chunks, H, TC, TC]
};

// ------------------------------------------------------------------------ token by token

template <typename T, int LPC, int EPL>
__global__ void __launch_bounds__(256) channel_scan_kernel(const ChannelArgs a, int tokens_staged) {
    constexpr int QPL = EPL / 4;
    constexpr int COLS = 8 * 32 / LPC;
    extern __shared__ __align__(16) float sm[];
    pdl_wait();
    pdl_trigger();
    const int r = blockIdx.z, head = blockIdx.y;
    const int t0 = a.row_start[r], n_new = a.row_start[r + 1] - t0;
    if (n_new <= 0 || n_new >= a.min_chunked) return;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int sub = lane % LPC;
    const int col0 = blockIdx.x * COLS;
    const int local = warp * (32 / LPC) + lane / LPC;
    const int col = col0 + local;
    const int N = a.N, V = a.V, H = a.H;
    const bool live = col < V;
    const T* q = reinterpret_cast<const T*>(a.q) + (int64_t)head * N;
    const T* k = reinterpret_cast<const T*>(a.k) + (int64_t)head * N;
    const T* v = reinterpret_cast<const T*>(a.v) + (int64_t)head * V;
    const float* lg = a.log_a + (int64_t)head * N;
    const float* bonus = a.u ? a.u + (int64_t)head * N : nullptr;
    float* st = a.state + (((int64_t)a.row_slot[r] * H + head) * V + (live ? col : 0)) * N;
    const bool quads = (N & 3) == 0;
    float S[EPL], U[EPL];
#pragma unroll
    for (int i = 0; i < QPL; ++i) {
        const int e = (i * LPC + sub) * 4;
        if (quads) {
            float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
            if (live && e < N) x = *reinterpret_cast<const float4*>(st + e);
            S[4 * i] = x.x; S[4 * i + 1] = x.y; S[4 * i + 2] = x.z; S[4 * i + 3] = x.w;
        } else {
#pragma unroll
            for (int w = 0; w < 4; ++w) S[4 * i + w] = (live && e + w < N) ? st[e + w] : 0.f;
        }
#pragma unroll
        for (int w = 0; w < 4; ++w) U[4 * i + w] = (bonus && e + w < N) ? bonus[e + w] : 0.f;
    }
    const int NP = (N + 3) / 4 * 4;            // staged rows, padded with zeros
    float* ks = sm;                            // [tokens_staged][NP]
    float* qs = ks + tokens_staged * NP;       // [tokens_staged][NP]
    float* as = qs + tokens_staged * NP;       // [tokens_staged][NP]: decays
    float* vs = as + tokens_staged * NP;       // [tokens_staged][COLS]
    for (int c0 = 0; c0 < n_new; c0 += tokens_staged) {
        const int nt = min(tokens_staged, n_new - c0);
        if (c0) __syncthreads();               // the previous tokens are no longer read
        if (quads && a.vec4) {                 // four elements of a row at a time
            const int per = N / 4;
#pragma unroll 2
            for (int i = tid; i < nt * per; i += 256) {
                const int t = i / per, e = (i - t * per) * 4;
                const int64_t n = t0 + c0 + t;
                const float4 l = load4(lg + n * H * N + e);
                *reinterpret_cast<float4*>(ks + t * NP + e) = load4(k + n * a.ldk + e);
                *reinterpret_cast<float4*>(qs + t * NP + e) = load4(q + n * a.ldq + e);
                *reinterpret_cast<float4*>(as + t * NP + e) =
                    make_float4(expf(l.x), expf(l.y), expf(l.z), expf(l.w));
            }
        } else {
            for (int i = tid; i < nt * NP; i += 256) {
                const int t = i / NP, e = i - t * NP;
                const int64_t n = t0 + c0 + t;
                ks[i] = e < N ? to_float(k[n * a.ldk + e]) : 0.f;
                qs[i] = e < N ? to_float(q[n * a.ldq + e]) : 0.f;
                as[i] = e < N ? expf(lg[n * H * N + e]) : 0.f;
            }
        }
        for (int i = tid; i < nt * COLS; i += 256) {
            const int t = i / COLS, j = col0 + i - t * COLS;
            vs[i] = j < V ? to_float(v[(int64_t)(t0 + c0 + t) * a.ldv + j]) : 0.f;
        }
        __syncthreads();
        for (int t = 0; t < nt; ++t) {
            const float value = vs[t * COLS + local];
            float part[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int i = 0; i < QPL; ++i) {
                const int e = (i * LPC + sub) * 4;
                if (e < NP) {
                    float kk[4], qq[4], aa[4];
                    *reinterpret_cast<float4*>(kk) = *reinterpret_cast<const float4*>(ks + t * NP + e);
                    *reinterpret_cast<float4*>(qq) = *reinterpret_cast<const float4*>(qs + t * NP + e);
                    *reinterpret_cast<float4*>(aa) = *reinterpret_cast<const float4*>(as + t * NP + e);
#pragma unroll
                    for (int w = 0; w < 4; ++w) {
                        const float kv = kk[w] * value, old = S[4 * i + w];
                        const float now = fmaf(aa[w], old, kv);
                        part[w] = fmaf(bonus ? fmaf(U[4 * i + w], kv, old) : now, qq[w], part[w]);
                        S[4 * i + w] = now;
                    }
                }
            }
            float acc = (part[0] + part[1]) + (part[2] + part[3]);
#pragma unroll
            for (int o = LPC / 2; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
            if (sub == 0 && live)
                a.out[(int64_t)(t0 + c0 + t) * H * V + (int64_t)head * V + col] = acc * a.scale;
        }
    }
    if (!live) return;
#pragma unroll
    for (int i = 0; i < QPL; ++i) {
        const int e = (i * LPC + sub) * 4;
        if (quads) {
            if (e < N)
                *reinterpret_cast<float4*>(st + e) =
                    make_float4(S[4 * i], S[4 * i + 1], S[4 * i + 2], S[4 * i + 3]);
        } else {
#pragma unroll
            for (int w = 0; w < 4; ++w)
                if (e + w < N) st[e + w] = S[4 * i + w];
        }
    }
}

// --------------------------------------------------------------------------- chunk kernels

struct Chunk { int row, t0, c0, n_new, nt; int64_t n0; };
__device__ __forceinline__ bool this_chunk(const ChannelArgs& a, Chunk& c) {
    if (!find_chunk(a.row_start, a.n_rows, a.min_chunked, blockIdx.x, c.row, c.t0, c.c0, c.n_new))
        return false;
    c.nt = min(TC, c.n_new - c.c0);
    c.n0 = c.t0 + c.c0;
    return true;
}

// The log decays of a block's BT tokens of one channel (0 beyond the chunk's tokens).
__device__ __forceinline__ void block_logs(const ChannelArgs& a, const Chunk& c, int head, int b, int e,
                                           float (&l)[BT]) {
    const float* lg = a.log_a + (c.n0 + b * BT) * a.H * a.N + (int64_t)head * a.N + e;
#pragma unroll
    for (int i = 0; i < BT; ++i)
        l[i] = (e < a.N && b * BT + i < c.nt) ? lg[(int64_t)i * a.H * a.N] : 0.f;
}

// Columns [v0, v0 + cols) of the chunk's values into shared memory (bfloat16, row stride ld), zeros
// beyond V and beyond the chunk's tokens.
__device__ __forceinline__ void stage_values(const ChannelArgs& a, bf16* dst, int ld, const bf16* v,
                                             int nt, int v0, int cols) {
    const int units = cols / 8;
    for (int i = threadIdx.x; i < TC * units; i += blockDim.x) {
        const int t = i / units, j = (i - t * units) * 8;
        alignas(16) bf16 x[8];
        const bf16* src = v + (int64_t)t * a.ldv + v0 + j;
        if (t < nt && v0 + j + 8 <= a.V && a.vec8) {
            *reinterpret_cast<uint4*>(x) = *reinterpret_cast<const uint4*>(src);
        } else {
#pragma unroll
            for (int w = 0; w < 8; ++w)
                x[w] = t < nt && v0 + j + w < a.V ? src[w] : __float2bfloat16_rn(0.f);
        }
        *reinterpret_cast<uint4*>(dst + t * ld + j) = *reinterpret_cast<const uint4*>(x);
    }
}
// The parts of one 32-bit number.
__device__ __forceinline__ void split1(float x, bf16* part) {
#pragma unroll
    for (int p = 0; p < PARTS; ++p) {
        part[p] = __float2bfloat16_rn(x);
        x -= __bfloat162float(part[p]);
    }
}

// A of one chunk and head; grid (slots, H), 256 threads.  The channels come in slabs of WB.
constexpr int WB = 64, LDW = WB + 4;
constexpr int W_FLOATS = 3 * TC * LDW + NB * WB + 3 * WB + WB;
template <typename T>
__global__ void __launch_bounds__(256, 3) channel_weights_kernel(const ChannelArgs a) {
    extern __shared__ __align__(16) float sm[];
    float* qs = sm;                       // [TC][LDW]
    float* ks = qs + TC * LDW;            // [TC][LDW]
    float* ps = ks + TC * LDW;            // [TC][LDW]: sums of log_a from the block's start on
    float* tot = ps + TC * LDW;           // [NB][WB]: the blocks' sums
    float* gaps = tot + NB * WB;          // [3][WB]: e^ of block 1's, block 2's, both blocks' sums
    float* us = gaps + 3 * WB;            // [WB]: u (or ones)
    pdl_wait();
    pdl_trigger();
    Chunk c;
    if (!this_chunk(a, c)) return;
    const int head = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int N = a.N, H = a.H;
    const T* q = reinterpret_cast<const T*>(a.q) + c.n0 * a.ldq + (int64_t)head * N;
    const T* k = reinterpret_cast<const T*>(a.k) + c.n0 * a.ldk + (int64_t)head * N;
    // Within blocks: tiles of 2 x 2 tokens, 28 below a block's diagonal, two threads a tile (even and
    // odd quads of channels): threads 0-223.  The tiles on the diagonal have one pair (t, t - 1) with
    // t odd, one thread each: threads 224-255.
    const bool single = tid >= 224;
    int near_t, near_s;                                      // the tile's first tokens
    if (single) {
        near_s = (tid - 224) * 2;
        near_t = near_s;
    } else {
        const int blk = tid / 56;
        int r = (tid - blk * 56) >> 1, t = 1;
        while (r >= t) { r -= t; ++t; }
        near_t = blk * BT + 2 * t;
        near_s = blk * BT + 2 * r;
    }
    float near[4] = {0.f, 0.f, 0.f, 0.f};
    // Between blocks: a warp per pair of blocks, tiles of 4 x 4 tokens, two threads a tile (four quads
    // of channels each in turn); warps 6 and 7 have the diagonal, a thread per token.
    const int far_tb = warp < 3 ? warp + 1 : warp == 3 ? 2 : 3;            // (1,0) (2,1) (3,2)
    const int far_sb = warp < 3 ? warp : warp == 4 ? 1 : 0;                // (2,0) (3,1) (3,0)
    const float* gap = warp < 3 || warp > 5 ? nullptr : gaps + (warp - 3) * WB;
    const int far_t = far_tb * BT + (lane >> 3), far_s = far_sb * BT + ((lane >> 1) & 3);
    float far[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i) far[i][0] = far[i][1] = far[i][2] = far[i][3] = 0.f;
    float own = 0.f;
    for (int e0 = 0; e0 < N; e0 += WB) {
        if (e0) __syncthreads();                             // the previous slab is no longer read
        const int b = tid / WB, j = tid % WB;                // a thread per (block, channel)
        {
            const int e = e0 + j;
            float l[BT];
            block_logs(a, c, head, b, e, l);
            float sum = 0.f;
#pragma unroll
            for (int i = 0; i < BT; ++i) {
                const int t = b * BT + i;
                const bool there = e < N && t < c.nt;
                sum += l[i];
                ps[t * LDW + j] = sum;
                qs[t * LDW + j] = there ? to_float(q[(int64_t)t * a.ldq + e]) : 0.f;
                ks[t * LDW + j] = there ? to_float(k[(int64_t)t * a.ldk + e]) : 0.f;
            }
            tot[b * WB + j] = sum;
            if (b == 0) us[j] = !a.u ? 1.f : e < N ? a.u[(int64_t)head * N + e] : 0.f;
        }
        __syncthreads();
        if (single) {
            const float* x = qs + (near_t + 1) * LDW;
            const float* y = ks + near_s * LDW;
            const float* E = ps + (near_t + (a.u ? 0 : 1)) * LDW;
            const float* L = ps + near_s * LDW;
#pragma unroll 4
            for (int i = 0; i < WB; i += 4) {
                const float4 xv = load4(x + i), yv = load4(y + i), ev = load4(E + i), lv = load4(L + i);
                near[2] = fmaf(xv.x * yv.x, __expf(ev.x - lv.x), near[2]);
                near[2] = fmaf(xv.y * yv.y, __expf(ev.y - lv.y), near[2]);
                near[2] = fmaf(xv.z * yv.z, __expf(ev.z - lv.z), near[2]);
                near[2] = fmaf(xv.w * yv.w, __expf(ev.w - lv.w), near[2]);
            }
        } else {
            const float* x = qs + near_t * LDW;
            const float* y = ks + near_s * LDW;
            const float* E = ps + (near_t - (a.u ? 1 : 0)) * LDW;
            const float* L = ps + near_s * LDW;
#pragma unroll 2
            for (int i = (tid & 1) * 4; i < WB; i += 8) {
                float xa[4], xb[4], ya[4], yb[4], ea[4], eb[4], la[4], lb[4];
                *reinterpret_cast<float4*>(xa) = load4(x + i);
                *reinterpret_cast<float4*>(xb) = load4(x + LDW + i);
                *reinterpret_cast<float4*>(ya) = load4(y + i);
                *reinterpret_cast<float4*>(yb) = load4(y + LDW + i);
                *reinterpret_cast<float4*>(ea) = load4(E + i);
                *reinterpret_cast<float4*>(eb) = load4(E + LDW + i);
                *reinterpret_cast<float4*>(la) = load4(L + i);
                *reinterpret_cast<float4*>(lb) = load4(L + LDW + i);
#pragma unroll
                for (int w = 0; w < 4; ++w) {
                    near[0] = fmaf(xa[w] * ya[w], __expf(ea[w] - la[w]), near[0]);
                    near[1] = fmaf(xa[w] * yb[w], __expf(ea[w] - lb[w]), near[1]);
                    near[2] = fmaf(xb[w] * ya[w], __expf(eb[w] - la[w]), near[2]);
                    near[3] = fmaf(xb[w] * yb[w], __expf(eb[w] - lb[w]), near[3]);
                }
            }
        }
        if (warp >= 6) {                                     // the diagonal
            const int t = tid - 192;
#pragma unroll 4
            for (int i = 0; i < WB; i += 4) {
                const float4 x = load4(qs + t * LDW + i), y = load4(ks + t * LDW + i), z = load4(us + i);
                own = fmaf(x.x * y.x, z.x, fmaf(x.y * y.y, z.y, fmaf(x.z * y.z, z.z,
                      fmaf(x.w * y.w, z.w, own))));
            }
        }
        __syncthreads();
        {   // q and k with their factors up to their blocks' borders, in place
            const float end = tot[b * WB + j];
            if (b > 0)
                gaps[(b - 1) * WB + j] = expf(b == 3 ? tot[WB + j] + tot[2 * WB + j] : end);
            float before = 0.f;
#pragma unroll
            for (int i = 0; i < BT; ++i) {
                const int at = (b * BT + i) * LDW + j;
                const float L = ps[at];
                qs[at] *= expf(a.u ? before : L);
                ks[at] *= expf(end - L);
                before = L;
            }
        }
        __syncthreads();
        if (warp < 6) {
            const float* x0 = qs + far_t * LDW;
            const float* y0 = ks + far_s * LDW;
#pragma unroll 1
            for (int i = 0; i < WB / 8; ++i) {
                const int at = ((i >> 2) * 8 + (lane & 1) * 4 + (i & 3)) * 4;
                float x[4][4], y[4][4];
#pragma unroll
                for (int r = 0; r < 4; ++r) {
                    *reinterpret_cast<float4*>(x[r]) = load4(x0 + 4 * r * LDW + at);
                    *reinterpret_cast<float4*>(y[r]) = load4(y0 + 4 * r * LDW + at);
                }
                if (gap) {
                    float f[4];
                    *reinterpret_cast<float4*>(f) = load4(gap + at);
#pragma unroll
                    for (int r = 0; r < 4; ++r)
#pragma unroll
                        for (int w = 0; w < 4; ++w) x[r][w] *= f[w];
                }
#pragma unroll
                for (int r = 0; r < 4; ++r)
#pragma unroll
                    for (int s = 0; s < 4; ++s)
#pragma unroll
                        for (int w = 0; w < 4; ++w) far[r][s] = fmaf(x[r][w], y[s][w], far[r][s]);
            }
        }
    }
    // (entries above the diagonal are never read)
    float* A = a.weights + ((int64_t)blockIdx.x * H + head) * TC * TC;
    if (!single) {
#pragma unroll
        for (int i = 0; i < 4; ++i) near[i] += __shfl_xor_sync(0xffffffffu, near[i], 1);
        if ((tid & 1) == 0) {
            *reinterpret_cast<float2*>(A + near_t * TC + near_s) = make_float2(near[0], near[1]);
            *reinterpret_cast<float2*>(A + (near_t + 1) * TC + near_s) = make_float2(near[2], near[3]);
        }
    } else {
        A[(near_t + 1) * TC + near_s] = near[2];
    }
    if (warp >= 6) {
        A[(tid - 192) * (TC + 1)] = own;
    } else {
#pragma unroll
        for (int r = 0; r < 4; ++r)
#pragma unroll
            for (int s = 0; s < 4; ++s) {
                const float sum = far[r][s] + __shfl_xor_sync(0xffffffffu, far[r][s], 1);
                if ((lane & 1) == (s & 1)) A[(far_t + 4 * r) * TC + far_s + 4 * s] = sum;
            }
    }
}

// dS of one chunk and head (32-bit rows): a tile of 64 key channels by 64 value columns; grid (slots, H, tiles),
// 128 threads, each 4 channels by 8 columns.
constexpr int ST_LD = 64 + 4;
template <typename T>
__global__ void __launch_bounds__(128) channel_state_kernel(const ChannelArgs a, int n_tiles) {
    __shared__ __align__(16) float ks[TC][ST_LD];          // e^{L_last - L_s} k_s
    __shared__ __align__(16) float vs[TC][ST_LD];
    __shared__ float tot[NB][64];
    pdl_wait();
    pdl_trigger();
    Chunk c;
    if (!this_chunk(a, c)) return;
    const int head = blockIdx.y, tid = threadIdx.x;
    const int N = a.N, V = a.V, H = a.H;
    const int e0 = (blockIdx.z % n_tiles) * 64, v0 = (blockIdx.z / n_tiles) * 64;
    const T* k = reinterpret_cast<const T*>(a.k) + c.n0 * a.ldk + (int64_t)head * N;
    const T* v = reinterpret_cast<const T*>(a.v) + c.n0 * a.ldv + (int64_t)head * V;
    const int j = tid & 63, e = e0 + j;
    float L[2][BT];
#pragma unroll
    for (int h = 0; h < 2; ++h) {                          // this thread's two blocks of tokens
        const int b = (tid >> 6) * 2 + h;
        block_logs(a, c, head, b, e, L[h]);
#pragma unroll
        for (int i = 1; i < BT; ++i) L[h][i] += L[h][i - 1];
        tot[b][j] = L[h][BT - 1];
    }
#pragma unroll 8
    for (int i = tid; i < TC * 64; i += 128) {
        const int t = i >> 6, col = v0 + (i & 63);
        vs[t][i & 63] = (t < c.nt && col < V) ? to_float(v[(int64_t)t * a.ldv + col]) : 0.f;
    }
    __syncthreads();
    float after = 0.f;
    for (int b = NB - 1; b > (tid >> 6) * 2 + 1; --b) after += tot[b][j];
#pragma unroll
    for (int h = 1; h >= 0; --h) {
        const int b = (tid >> 6) * 2 + h;
        const float end = L[h][BT - 1];
#pragma unroll
        for (int i = 0; i < BT; ++i) {
            const int t = b * BT + i;
            ks[t][j] = (e < N && t < c.nt)
                ? to_float(k[(int64_t)t * a.ldk + e]) * expf(after + (end - L[h][i])) : 0.f;
        }
        after += end;
    }
    if (v0 == 0 && tid < 64 && e < N)
        a.decay[((int64_t)blockIdx.x * H + head) * N + e] = after;   // (threads 0-63 have met every block)
    __syncthreads();
    const int x = (tid & 15) * 4, y = (tid >> 4) * 8;
    float acc[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll 4
    for (int t = 0; t < TC; ++t) {
        float kk[4], vv[8];
        *reinterpret_cast<float4*>(kk) = load4(&ks[t][x]);
        *reinterpret_cast<float4*>(vv) = load4(&vs[t][y]);
        *reinterpret_cast<float4*>(vv + 4) = load4(&vs[t][y + 4]);
#pragma unroll
        for (int i = 0; i < 8; ++i)
#pragma unroll
            for (int w = 0; w < 4; ++w) acc[i][w] = fmaf(vv[i], kk[w], acc[i][w]);
    }
    float* dst = a.dS + ((int64_t)blockIdx.x * H + head) * V * N;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        if (v0 + y + i >= V) break;
        float* d = dst + (int64_t)(v0 + y + i) * N + e0 + x;
        if ((N & 3) == 0) {
            if (e0 + x < N)
                *reinterpret_cast<float4*>(d) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
        } else {
#pragma unroll
            for (int w = 0; w < 4; ++w)
                if (e0 + x + w < N) d[w] = acc[i][w];
        }
    }
}

// The states at the chunks' starts, in place of the chunks' own dS, and the row's final state into
// its slot.  A thread per W elements (4 where N allows it, else 1); grid (ceil(V N / W / 256), H, rows).
constexpr int PASS_AHEAD = 8;
template <int W>
__global__ void __launch_bounds__(256) channel_pass_kernel(const ChannelArgs a) {
    pdl_wait();
    pdl_trigger();
    struct alignas(W * 4) Part { float x[W]; };
    const int r = blockIdx.z, head = blockIdx.y;
    const int t0 = a.row_start[r], n_new = a.row_start[r + 1] - t0;
    if (n_new <= 0 || n_new < a.min_chunked) return;
    const int64_t size = (int64_t)a.V * a.N;
    const int64_t e = ((int64_t)blockIdx.x * 256 + threadIdx.x) * W;
    if (e >= size) return;
    const int n_chunks = (n_new + TC - 1) / TC;
    const int64_t slot0 = t0 / TC + r;
    float* d = a.dS + (slot0 * a.H + head) * size + e;
    const float* dec = a.decay + (slot0 * a.H + head) * a.N + e % a.N;
    const int64_t step = (int64_t)a.H * size, dstep = (int64_t)a.H * a.N;
    float* home = a.state + ((int64_t)a.row_slot[r] * a.H + head) * size + e;
    Part S = *reinterpret_cast<const Part*>(home);
    for (int c0 = 0; c0 < n_chunks; c0 += PASS_AHEAD) {
        Part x[PASS_AHEAD], f[PASS_AHEAD];
#pragma unroll
        for (int i = 0; i < PASS_AHEAD; ++i)
            if (c0 + i < n_chunks) {
                x[i] = *reinterpret_cast<const Part*>(d + (c0 + i) * step);
                f[i] = *reinterpret_cast<const Part*>(dec + (c0 + i) * dstep);
            }
#pragma unroll
        for (int i = 0; i < PASS_AHEAD; ++i)
            if (c0 + i < n_chunks) {
                *reinterpret_cast<Part*>(d + (c0 + i) * step) = S;
#pragma unroll
                for (int w = 0; w < W; ++w) S.x[w] = fmaf(expf(f[i].x[w]), S.x[w], x[i].x[w]);
            }
    }
    *reinterpret_cast<Part*>(home) = S;
}

// The read-outs of one chunk and head (32-bit rows), 64 value columns; grid (slots, H, ceil(V / 64)), 128 threads:
// thread (tg, vg) has the tokens 8 tg .. 8 tg + 7 and the columns vg, vg + 16, vg + 32, vg + 48.
constexpr int OB = 32, OLD = OB + 4;                        // channels of a slab
template <typename T>
__global__ void __launch_bounds__(128) channel_out_kernel(const ChannelArgs a) {
    // the queries' and the state's slab; later the weights and the values
    __shared__ __align__(16) float buf[2 * TC * ST_LD];
    __shared__ float tot[NB][OB];
    float* qs = buf;                   // [TC][OLD]: e^{E_t} q_t
    float* ss = buf + TC * OLD;        // [64][OLD]: S0's columns
    float* ws = buf;                   // [TC][ST_LD]
    float* vs = buf + TC * ST_LD;      // [TC][ST_LD]
    pdl_wait();
    pdl_trigger();
    Chunk c;
    if (!this_chunk(a, c)) return;
    const int head = blockIdx.y, v0 = blockIdx.z * 64, tid = threadIdx.x;
    const int N = a.N, V = a.V, H = a.H;
    const T* q = reinterpret_cast<const T*>(a.q) + c.n0 * a.ldq + (int64_t)head * N;
    const T* v = reinterpret_cast<const T*>(a.v) + c.n0 * a.ldv + (int64_t)head * V;
    const float* s0 = a.dS + (((int64_t)blockIdx.x * H + head) * V + v0) * N;
    const int tg = tid >> 4, vg = tid & 15;
    float o[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    for (int e0 = 0; e0 < N; e0 += OB) {
        if (e0) __syncthreads();                             // the previous slab is no longer read
        const int b = tid / OB, j = tid % OB, e = e0 + j;    // 16 tokens of one channel
        float l[BT];
        block_logs(a, c, head, b, e, l);
#pragma unroll
        for (int i = 1; i < BT; ++i) l[i] += l[i - 1];
        tot[b][j] = l[BT - 1];
#pragma unroll 8
        for (int i = tid; i < 64 * OB; i += 128) {
            const int col = i / OB, ee = e0 + i % OB;
            ss[col * OLD + i % OB] = (v0 + col < V && ee < N) ? s0[(int64_t)col * N + ee] : 0.f;
        }
        __syncthreads();
        float before = 0.f;
        for (int p = 0; p < b; ++p) before += tot[p][j];
#pragma unroll
        for (int i = 0; i < BT; ++i) {
            const int t = b * BT + i;
            const float E = before + (a.u ? (i ? l[i - 1] : 0.f) : l[i]);
            qs[t * OLD + j] = (e < N && t < c.nt) ? to_float(q[(int64_t)t * a.ldq + e]) * expf(E) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int n = 0; n < OB; n += 4) {
            float4 sv[4];
#pragma unroll
            for (int w = 0; w < 4; ++w) sv[w] = load4(ss + (vg + 16 * w) * OLD + n);
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const float4 x = load4(qs + (tg * 8 + i) * OLD + n);
#pragma unroll
                for (int w = 0; w < 4; ++w)
                    o[i][w] = fmaf(x.x, sv[w].x, fmaf(x.y, sv[w].y, fmaf(x.z, sv[w].z,
                              fmaf(x.w, sv[w].w, o[i][w]))));
            }
        }
    }
    __syncthreads();
    const float* A = a.weights + ((int64_t)blockIdx.x * H + head) * TC * TC;
#pragma unroll 4
    for (int i = tid; i < TC * TC / 4; i += 128) {
        const int t = i / (TC / 4), s = (i % (TC / 4)) * 4;
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
        if (s <= t) {
            x = load4(A + t * TC + s);
            if (s + 1 > t) x.y = 0.f;
            if (s + 2 > t) x.z = 0.f;
            if (s + 3 > t) x.w = 0.f;
        }
        *reinterpret_cast<float4*>(ws + t * ST_LD + s) = x;
    }
#pragma unroll 8
    for (int i = tid; i < TC * 64; i += 128) {
        const int t = i >> 6, col = v0 + (i & 63);
        vs[t * ST_LD + (i & 63)] = (t < c.nt && col < V) ? to_float(v[(int64_t)t * a.ldv + col]) : 0.f;
    }
    __syncthreads();
    const int s_end = (tid >> 5) * 16 + 16;                  // this warp's tokens see no later ones
    for (int s = 0; s < s_end; s += 4) {
        float vv[4][4];
#pragma unroll
        for (int u = 0; u < 4; ++u)
#pragma unroll
            for (int w = 0; w < 4; ++w) vv[u][w] = vs[(s + u) * ST_LD + vg + 16 * w];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const float4 x = load4(ws + (tg * 8 + i) * ST_LD + s);
#pragma unroll
            for (int w = 0; w < 4; ++w)
                o[i][w] = fmaf(x.x, vv[0][w], fmaf(x.y, vv[1][w], fmaf(x.z, vv[2][w],
                          fmaf(x.w, vv[3][w], o[i][w]))));
        }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int t = tg * 8 + i;
        if (t >= c.nt) break;
        float* dst = a.out + (c.n0 + t) * H * V + (int64_t)head * V + v0;
#pragma unroll
        for (int w = 0; w < 4; ++w)
            if (v0 + vg + 16 * w < V) dst[vg + 16 * w] = o[i][w] * a.scale;
    }
}

// dS of one chunk and head on the tensor cores (bfloat16 rows): a tile of 64 key channels by 128 value
// columns; grid (slots, H, tiles), 256 threads, a warp per 16 columns.
constexpr int MV = 128, MLD = 64 + 8, MLDV = MV + 8;
constexpr size_t STATE_MMA_SMEM = ((size_t)PARTS * TC * MLD + (size_t)TC * MLDV) * sizeof(bf16);
__global__ void __launch_bounds__(256) channel_state_mma_kernel(const ChannelArgs a, int n_tiles) {
    extern __shared__ __align__(16) unsigned char raw[];
    __shared__ float tot[NB][64];
    bf16* ks = reinterpret_cast<bf16*>(raw);               // [PARTS][TC][MLD]: e^{L_last - L_s} k_s
    bf16* vs = ks + PARTS * TC * MLD;                      // [TC][MLDV]
    pdl_wait();
    pdl_trigger();
    Chunk c;
    if (!this_chunk(a, c)) return;
    const int head = blockIdx.y, tid = threadIdx.x;
    const int N = a.N, V = a.V, H = a.H;
    const int e0 = (blockIdx.z % n_tiles) * 64, v0 = (blockIdx.z / n_tiles) * MV;
    const bf16* k = reinterpret_cast<const bf16*>(a.k) + c.n0 * a.ldk + (int64_t)head * N;
    const bf16* v = reinterpret_cast<const bf16*>(a.v) + c.n0 * a.ldv + (int64_t)head * V;
    const int j = tid & 63, b = tid >> 6, e = e0 + j;
    float L[BT];
    block_logs(a, c, head, b, e, L);
    bf16 kk[BT];
#pragma unroll
    for (int i = 0; i < BT; ++i)
        kk[i] = (e < N && b * BT + i < c.nt) ? k[(int64_t)(b * BT + i) * a.ldk + e]
                                             : __float2bfloat16_rn(0.f);
    stage_values(a, vs, MLDV, v, c.nt, v0, MV);
#pragma unroll
    for (int i = 1; i < BT; ++i) L[i] += L[i - 1];
    const float end = L[BT - 1];
    tot[b][j] = end;
    __syncthreads();
    float after = 0.f;
    for (int p = NB - 1; p > b; --p) after += tot[p][j];
#pragma unroll
    for (int i = 0; i < BT; ++i) {
        bf16 part[PARTS];
        split1(__bfloat162float(kk[i]) * expf(after + (end - L[i])), part);
#pragma unroll
        for (int p = 0; p < PARTS; ++p) ks[(p * TC + b * BT + i) * MLD + j] = part[p];
    }
    if (v0 == 0 && b == 0 && e < N) a.decay[((int64_t)blockIdx.x * H + head) * N + e] = after + end;
    __syncthreads();
    const int warp = tid >> 5, lane = tid & 31;
    if (v0 + warp * 16 >= V) return;
    // A[m = column][k = token] from [token][column]: transposed 8 x 8 blocks in the order
    // (m 0-7, k 0-7), (m 8-15, k 0-7), (m 0-7, k 8-15), (m 8-15, k 8-15)
    uint32_t af[TC / 16][4];
    const int blk = lane >> 3;
#pragma unroll
    for (int kt = 0; kt < TC / 16; ++kt)
        ldsm4_t(af[kt], smem_addr(vs + (kt * 16 + (blk >> 1) * 8 + (lane & 7)) * MLDV + warp * 16 +
                                  (blk & 1) * 8));
    float acc[8][4];
#pragma unroll
    for (int u = 0; u < 8; ++u) acc[u][0] = acc[u][1] = acc[u][2] = acc[u][3] = 0.f;
#pragma unroll
    for (int p = PARTS - 1; p >= 0; --p)                   // small parts first
#pragma unroll
        for (int kt = 0; kt < TC / 16; ++kt)
#pragma unroll
            for (int u = 0; u < 8; u += 2) {
                uint32_t bf[4];
                ldsm4_t(bf, smem_addr(ks + (p * TC + kt * 16 + (lane & 15)) * MLD + u * 8 +
                                      (lane >> 4) * 8));
                mma_bf16(acc[u], af[kt], bf);
                mma_bf16(acc[u + 1], af[kt], bf + 2);
            }
    float* dst = a.dS + ((int64_t)blockIdx.x * H + head) * V * N;
#pragma unroll
    for (int u = 0; u < 8; ++u)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            const int m = v0 + warp * 16 + (lane >> 2) + 8 * h, n = e0 + u * 8 + (lane & 3) * 2;
            if (m >= V || n >= N) continue;
            float* d = dst + (int64_t)m * N + n;
            if ((N & 1) == 0) {
                *reinterpret_cast<float2*>(d) = make_float2(acc[u][2 * h], acc[u][2 * h + 1]);
            } else {
                d[0] = acc[u][2 * h];
                if (n + 1 < N) d[1] = acc[u][2 * h + 1];
            }
        }
}

// The read-outs of one chunk and head on the tensor cores (bfloat16 rows), 64 value columns; grid
// (slots, H, ceil(V / 64)), 256 threads: warps w and w + 4 have the chunk's tokens 16 w .. 16 w + 15,
// and half of the columns each.  Queries and state go through shared memory in slabs of 64 channels.
constexpr size_t OUT_MMA_SMEM = ((size_t)2 * PARTS * TC * MLD + (size_t)TC * MLD) * sizeof(bf16);
__global__ void __launch_bounds__(256, 3) channel_out_mma_kernel(const ChannelArgs a) {
    extern __shared__ __align__(16) unsigned char raw[];
    __shared__ float tot[NB][64];
    bf16* qs = reinterpret_cast<bf16*>(raw);               // [PARTS][TC][MLD]: e^{E_t} q_t
    bf16* ss = qs + PARTS * TC * MLD;                      // [PARTS][64][MLD]: S0's columns
    bf16* vs = ss + PARTS * TC * MLD;                      // [TC][MLD]
    pdl_wait();
    pdl_trigger();
    Chunk c;
    if (!this_chunk(a, c)) return;
    const int head = blockIdx.y, v0 = blockIdx.z * 64, tid = threadIdx.x;
    const int warp = tid >> 5, lane = tid & 31;
    const int N = a.N, V = a.V, H = a.H;
    const bf16* q = reinterpret_cast<const bf16*>(a.q) + c.n0 * a.ldq + (int64_t)head * N;
    const bf16* v = reinterpret_cast<const bf16*>(a.v) + c.n0 * a.ldv + (int64_t)head * V;
    const float* s0 = a.dS + (((int64_t)blockIdx.x * H + head) * V + v0) * N;
    stage_values(a, vs, MLD, v, c.nt, v0, 64);
    const int m0 = (warp & 3) * 16, n0 = (warp >> 2) * 32;
    float o[4][4];
#pragma unroll
    for (int u = 0; u < 4; ++u) o[u][0] = o[u][1] = o[u][2] = o[u][3] = 0.f;
    const int j = tid & 63, b = tid >> 6;
    for (int e0 = 0; e0 < N; e0 += 64) {
        const int e = e0 + j;
        float L[BT];
        block_logs(a, c, head, b, e, L);
        bf16 qq[BT];
#pragma unroll
        for (int i = 0; i < BT; ++i)
            qq[i] = (e < N && b * BT + i < c.nt) ? q[(int64_t)(b * BT + i) * a.ldq + e]
                                                 : __float2bfloat16_rn(0.f);
        const int se = (tid & 15) * 4;
        float4 sx[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int col = (tid >> 4) + i * 16;
            sx[i] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (v0 + col >= V || e0 + se >= N) continue;
            const float* at = s0 + (int64_t)col * N + e0 + se;
            if ((N & 3) == 0) {
                sx[i] = load4(at);
            } else {
                sx[i].x = at[0];
                if (e0 + se + 1 < N) sx[i].y = at[1];
                if (e0 + se + 2 < N) sx[i].z = at[2];
                if (e0 + se + 3 < N) sx[i].w = at[3];
            }
        }
#pragma unroll
        for (int i = 1; i < BT; ++i) L[i] += L[i - 1];
        if (e0) __syncthreads();                           // the previous slab is no longer read
        tot[b][j] = L[BT - 1];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            uint32_t lo[PARTS], hi[PARTS];
            split2(sx[i].x, sx[i].y, lo);
            split2(sx[i].z, sx[i].w, hi);
#pragma unroll
            for (int p = 0; p < PARTS; ++p)
                *reinterpret_cast<uint2*>(ss + (p * TC + (tid >> 4) + i * 16) * MLD + se) =
                    make_uint2(lo[p], hi[p]);
        }
        __syncthreads();
        float before = 0.f;
        for (int p = 0; p < b; ++p) before += tot[p][j];
#pragma unroll
        for (int i = 0; i < BT; ++i) {
            const float E = before + (a.u ? (i ? L[i - 1] : 0.f) : L[i]);
            bf16 part[PARTS];
            split1(__bfloat162float(qq[i]) * expf(E), part);
#pragma unroll
            for (int p = 0; p < PARTS; ++p) qs[(p * TC + b * BT + i) * MLD + j] = part[p];
        }
        __syncthreads();
        const int steps = (min(64, N - e0) + 15) / 16;
        for (int kt = 0; kt < steps; ++kt) {
            uint32_t af[PARTS][4];
#pragma unroll
            for (int p = 0; p < PARTS; ++p)
                ldsm4(af[p], smem_addr(qs + (p * TC + m0 + (lane & 15)) * MLD + kt * 16 + (lane >> 4) * 8));
#pragma unroll
            for (int u = 0; u < 4; u += 2) {
                uint32_t bf[PARTS][4];
#pragma unroll
                for (int p = 0; p < PARTS; ++p)
                    ldsm4(bf[p], smem_addr(ss + (p * TC + n0 + (u + (lane >> 4)) * 8 + (lane & 7)) * MLD +
                                           kt * 16 + ((lane >> 3) & 1) * 8));
#pragma unroll
                for (int sum = PARTS - 1; sum >= 0; --sum)  // parts p of q and sum - p of S0
#pragma unroll
                    for (int p = 0; p <= sum; ++p) {
                        mma_bf16(o[u], af[p], bf[sum - p]);
                        mma_bf16(o[u + 1], af[p], bf[sum - p] + 2);
                    }
            }
        }
    }
    __syncthreads();
    // the weights, split, in the queries' place
    const float* A = a.weights + ((int64_t)blockIdx.x * H + head) * TC * TC;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = (tid >> 4) + i * 16, s = (tid & 15) * 4;
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
        if (s <= t) {
            x = load4(A + t * TC + s);
            if (s + 1 > t) x.y = 0.f;
            if (s + 2 > t) x.z = 0.f;
            if (s + 3 > t) x.w = 0.f;
        }
        uint32_t lo[PARTS], hi[PARTS];
        split2(x.x, x.y, lo);
        split2(x.z, x.w, hi);
#pragma unroll
        for (int p = 0; p < PARTS; ++p)
            *reinterpret_cast<uint2*>(qs + (p * TC + t) * MLD + s) = make_uint2(lo[p], hi[p]);
    }
    __syncthreads();
    for (int kt = 0; kt * 16 <= m0; ++kt) {                // tokens s of 16
        uint32_t af[PARTS][4];
#pragma unroll
        for (int p = 0; p < PARTS; ++p)
            ldsm4(af[p], smem_addr(qs + (p * TC + m0 + (lane & 15)) * MLD + kt * 16 + (lane >> 4) * 8));
#pragma unroll
        for (int u = 0; u < 4; u += 2) {
            uint32_t bf[4];
            ldsm4_t(bf, smem_addr(vs + (kt * 16 + (lane & 15)) * MLD + n0 + u * 8 + (lane >> 4) * 8));
#pragma unroll
            for (int p = PARTS - 1; p >= 0; --p) {
                mma_bf16(o[u], af[p], bf);
                mma_bf16(o[u + 1], af[p], bf + 2);
            }
        }
    }
#pragma unroll
    for (int u = 0; u < 4; ++u)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            const int t = m0 + (lane >> 2) + 8 * h, col = v0 + n0 + u * 8 + (lane & 3) * 2;
            if (t >= c.nt || col >= V) continue;
            float* d = a.out + (c.n0 + t) * H * V + (int64_t)head * V + col;
            const float x = o[u][2 * h] * a.scale, y = o[u][2 * h + 1] * a.scale;
            if ((V & 1) == 0) {
                *reinterpret_cast<float2*>(d) = make_float2(x, y);
            } else {
                d[0] = x;
                if (col + 1 < V) d[1] = y;
            }
        }
}

template <typename T>
static cudaError_t launch_chunks(const ChannelArgs& a, int n_tokens, cudaStream_t stream) {
    const int slots = n_tokens / TC + a.n_rows + 1;
    const int nt = (a.N + 63) / 64, vt = (a.V + 63) / 64;
    const size_t smem = (size_t)W_FLOATS * sizeof(float);
    constexpr bool TENSOR = sizeof(T) == 2;
    static bool ready = false;
    if (!ready) {
        const cudaFuncAttribute attr = cudaFuncAttributeMaxDynamicSharedMemorySize;
        cudaError_t e = cudaFuncSetAttribute(channel_weights_kernel<T>, attr, (int)smem);
        if (e == cudaSuccess && TENSOR)
            e = cudaFuncSetAttribute(channel_out_mma_kernel, attr, (int)OUT_MMA_SMEM);
        if (e != cudaSuccess) return e;
        ready = true;
    }
    cudaError_t e = sllm_launch_pdl(channel_weights_kernel<T>, dim3(slots, a.H), dim3(256), smem,
                                    stream, a);
    if (e != cudaSuccess) return e;
    if (TENSOR)
        e = sllm_launch_pdl(channel_state_mma_kernel, dim3(slots, a.H, nt * ((a.V + MV - 1) / MV)),
                            dim3(256), STATE_MMA_SMEM, stream, a, nt);
    else
        e = sllm_launch_pdl(channel_state_kernel<float>, dim3(slots, a.H, nt * vt), dim3(128), 0, stream,
                            a, nt);
    if (e != cudaSuccess) return e;
    const int64_t size = (int64_t)a.V * a.N;
    if ((a.N & 3) == 0)
        e = sllm_launch_pdl(channel_pass_kernel<4>, dim3((unsigned)((size / 4 + 255) / 256), a.H, a.n_rows),
                            dim3(256), 0, stream, a);
    else
        e = sllm_launch_pdl(channel_pass_kernel<1>, dim3((unsigned)((size + 255) / 256), a.H, a.n_rows),
                            dim3(256), 0, stream, a);
    if (e != cudaSuccess) return e;
    if (TENSOR)
        return sllm_launch_pdl(channel_out_mma_kernel, dim3(slots, a.H, vt), dim3(256), OUT_MMA_SMEM,
                               stream, a);
    return sllm_launch_pdl(channel_out_kernel<float>, dim3(slots, a.H, vt), dim3(128), 0, stream, a);
}

}  // namespace sllm

using namespace sllm;

SLLM_EXPORT int sllm_channel_scan_chunk() { return TC; }

// q, k: [n_tokens, >= H N], v: [n_tokens, >= H V] (dtype), log_a: float [n_tokens, H N]; u: float
// [H N] or null; state: float [slots, H, V, N]; out: float [n_tokens, H V].  chunked: rows of at
// least min_chunked tokens take the chunk kernels, with the scratch dS float [n_tokens / 64 + n_rows
// + 1, H, V, N], decay float [the same, H, N] and weights float [the same, H, 64, 64]; else every row
// is walked token by token.  shortest / longest: bounds of the tokens a row brings.
SLLM_EXPORT int sllm_channel_scan(const void* q, int64_t ldq, const void* k, int64_t ldk,
                                  const void* v, int64_t ldv, const float* log_a, const float* u,
                                  float* state, const int* row_start, const int* row_slot, float* out,
                                  float scale, int n_tokens, int n_rows, int H, int N, int V,
                                  int chunked, int min_chunked, int shortest, int longest, float* dS,
                                  float* decay, float* weights, int dtype, cudaStream_t stream) {
    if (n_tokens <= 0 || n_rows <= 0) return 0;
    if (H < 1 || N < 1 || N > 1024 || V < 1 || ldq < (int64_t)H * N || ldk < (int64_t)H * N ||
        ldv < (int64_t)H * V || H > 65535 || n_rows > 65535 || dtype < 0 || dtype > 1)
        return (int)cudaErrorInvalidValue;
    const int vec4 = !((ldq | ldk | N) & 3) &&
                     !(((uintptr_t)q | (uintptr_t)k | (uintptr_t)log_a) & 15);
    const int vec8 = !((ldv | V) & 7) && !((uintptr_t)v & 15);
    ChannelArgs a = {q, ldq, k, ldk, v, ldv, log_a, u, state, row_start, row_slot, out, scale,
                     H, N, V, vec4, vec8, 0x7fffffff, n_rows, dS, decay, weights};
    if ((N & 3) == 0 && ((uintptr_t)state & 15)) return (int)cudaErrorInvalidValue;
    if (chunked) {
        if (!dS || !decay || !weights || min_chunked < 1 ||
            (((uintptr_t)dS | (uintptr_t)decay | (uintptr_t)weights) & 15) ||
            (int64_t)((N + 63) / 64) * ((V + 63) / 64) > 65535)
            return (int)cudaErrorInvalidValue;
        a.min_chunked = min_chunked;
        const cudaError_t e = dtype == 0 ? launch_chunks<float>(a, n_tokens, stream)
                                         : launch_chunks<bf16>(a, n_tokens, stream);
        if (e != cudaSuccess) return (int)e;
    }
    const int NP = (N + 3) / 4 * 4;
    int limit = longest > 0 ? longest : 32;
    if (chunked && limit > min_chunked - 1) limit = min_chunked - 1;
    if (limit < 1 || (chunked && shortest >= min_chunked)) return 0;   // nothing left
#define SLLM_SCAN(T, LPC, EPL)                                                                     \
    do {                                                                                           \
        constexpr int cols = 8 * 32 / LPC;                                                         \
        const int per = (3 * NP + cols) * (int)sizeof(float);                                      \
        int staged = 47 * 1024 / per;                                                              \
        if (staged > 32) staged = 32;                                                              \
        if (staged > limit) staged = limit;                                                        \
        return (int)sllm_launch_pdl(channel_scan_kernel<T, LPC, EPL>,                              \
                                    dim3((V + cols - 1) / cols, H, n_rows), dim3(256),             \
                                    (size_t)staged * per, stream, a, staged);                      \
    } while (0)
#define SLLM_SCAN_N(T)                                                                             \
    do {                                                                                           \
        if (N <= 32) SLLM_SCAN(T, 8, 4);                                                           \
        if (N <= 64) SLLM_SCAN(T, 8, 8);                                                           \
        if (N <= 128) SLLM_SCAN(T, 8, 16);                                                         \
        if (N <= 256) SLLM_SCAN(T, 8, 32);                                                         \
        if (N <= 512) SLLM_SCAN(T, 32, 16);                                                        \
        SLLM_SCAN(T, 32, 32);                                                                      \
    } while (0)
    if (dtype == 0) SLLM_SCAN_N(float);
    SLLM_SCAN_N(bf16);
#undef SLLM_SCAN_N
#undef SLLM_SCAN
}
