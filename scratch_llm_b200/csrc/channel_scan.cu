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
// go to q and k beforehand.  Everything is 32-bit fused multiply-adds on the CUDA cores: the operands
// of every product are 32-bit (decayed keys and queries, the state), and the sizes are small, so the
// splitting of both operands into bfloat16 parts would cost more than the products.
#include "scan_chunks.cuh"

namespace sllm {

constexpr int BT = 16;              // tokens of a block inside a chunk
constexpr int NB = TC / BT;
typedef __nv_bfloat16 bf16;

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

// A of one chunk and head; grid (slots, H), 256 threads.  The channels come in slabs of WB.
constexpr int WB = 64, LDW = WB + 4;
constexpr int W_FLOATS = 3 * TC * LDW + 2 * NB * WB;
template <typename T>
__global__ void __launch_bounds__(256) channel_weights_kernel(const ChannelArgs a) {
    extern __shared__ __align__(16) float sm[];
    float* qs = sm;                       // [TC][LDW]
    float* ks = qs + TC * LDW;            // [TC][LDW]
    float* ps = ks + TC * LDW;            // [TC][LDW]: sums of log_a from the block's start on
    float* tot = ps + TC * LDW;           // [NB][WB]: the blocks' sums
    float* us = tot + NB * WB;            // [WB]: u (or ones)
    pdl_wait();
    pdl_trigger();
    Chunk c;
    if (!this_chunk(a, c)) return;
    const int head = blockIdx.y, tid = threadIdx.x;
    const int N = a.N, H = a.H;
    const T* q = reinterpret_cast<const T*>(a.q) + c.n0 * a.ldq + (int64_t)head * N;
    const T* k = reinterpret_cast<const T*>(a.k) + c.n0 * a.ldk + (int64_t)head * N;
    // within blocks: the strict lower triangles' pairs, two per thread; pair p of a block is (t, s)
    // with p = t (t - 1) / 2 + s
    constexpr int PAIRS = BT * (BT - 1) / 2;                 // 120
    int pt[2], psrc[2];
    float pair[2] = {0.f, 0.f};
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int p = tid + i * 256, b = p / PAIRS;
        int r = p - b * PAIRS, t = 1;
        while (r >= t) { r -= t; ++t; }
        pt[i] = b * BT + t;
        psrc[i] = b * BT + r;
        if (b >= NB) pt[i] = -1;
    }
    // between blocks: 64 threads a pair of blocks, 2 x 2 tokens a thread; the six pairs of blocks are
    // (1,0) (2,1) (3,2) (2,0) and (3,1) (3,0), the second two taken by the first two groups
    const int group = tid >> 6, in = tid & 63, ti = (in >> 3) * 2, si = (in & 7) * 2;
    float far[2][4];
#pragma unroll
    for (int i = 0; i < 2; ++i) far[i][0] = far[i][1] = far[i][2] = far[i][3] = 0.f;
    const int tb[2] = {group < 3 ? group + 1 : 2, 3};
    const int sb[2] = {group < 3 ? group : 0, group == 0 ? 1 : 0};
    float own = 0.f;                                         // the diagonal: four threads a token
    for (int e0 = 0; e0 < N; e0 += WB) {
        if (e0) __syncthreads();                             // the previous slab is no longer read
        {   // a thread per (block, channel): 16 tokens
            const int b = tid / WB, j = tid % WB, e = e0 + j;
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
        {   // the diagonal
            const int t = tid >> 2, part = tid & 3;
#pragma unroll
            for (int i = 0; i < WB / 16; ++i) {
                const int j = (part + 4 * i) * 4;
                const float4 x = load4(qs + t * LDW + j), y = load4(ks + t * LDW + j), z = load4(us + j);
                own = fmaf(x.x * y.x, z.x, fmaf(x.y * y.y, z.y, fmaf(x.z * y.z, z.z,
                      fmaf(x.w * y.w, z.w, own))));
            }
        }
#pragma unroll
        for (int i = 0; i < 2; ++i) {                        // pairs of a block
            if (pt[i] < 0) continue;
            const float* x = qs + pt[i] * LDW;
            const float* y = ks + psrc[i] * LDW;
            const float* Et = ps + (pt[i] - (a.u ? 1 : 0)) * LDW;
            const float* Ls = ps + psrc[i] * LDW;
            float acc = pair[i];
#pragma unroll 4
            for (int j = 0; j < WB; j += 4) {
                const float4 xv = load4(x + j), yv = load4(y + j), ev = load4(Et + j), lv = load4(Ls + j);
                acc = fmaf(xv.x * yv.x, __expf(ev.x - lv.x), acc);
                acc = fmaf(xv.y * yv.y, __expf(ev.y - lv.y), acc);
                acc = fmaf(xv.z * yv.z, __expf(ev.z - lv.z), acc);
                acc = fmaf(xv.w * yv.w, __expf(ev.w - lv.w), acc);
            }
            pair[i] = acc;
        }
        __syncthreads();
        {   // q and k with their factors up to their blocks' borders, in place
            const int b = tid / WB, j = tid % WB;
            const float end = tot[b * WB + j];
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
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            if (i == 1 && group >= 2) break;
            const float* x0 = qs + (tb[i] * BT + ti) * LDW;
            const float* y0 = ks + (sb[i] * BT + si) * LDW;
            const int gap = tb[i] - sb[i] - 1;               // whole blocks in between
            float s00 = far[i][0], s01 = far[i][1], s10 = far[i][2], s11 = far[i][3];
#pragma unroll 4
            for (int j = 0; j < WB; j += 4) {
                float xa[4], xb[4], ya[4], yb[4];
                *reinterpret_cast<float4*>(xa) = load4(x0 + j);
                *reinterpret_cast<float4*>(xb) = load4(x0 + LDW + j);
                *reinterpret_cast<float4*>(ya) = load4(y0 + j);
                *reinterpret_cast<float4*>(yb) = load4(y0 + LDW + j);
                if (gap > 0) {
                    float f[4];
                    *reinterpret_cast<float4*>(f) = load4(tot + (sb[i] + 1) * WB + j);
                    if (gap > 1) {
                        const float4 g = load4(tot + (sb[i] + 2) * WB + j);
                        f[0] += g.x; f[1] += g.y; f[2] += g.z; f[3] += g.w;
                    }
#pragma unroll
                    for (int w = 0; w < 4; ++w) {
                        f[w] = __expf(f[w]);
                        xa[w] *= f[w];
                        xb[w] *= f[w];
                    }
                }
#pragma unroll
                for (int w = 0; w < 4; ++w) {
                    s00 = fmaf(xa[w], ya[w], s00);
                    s01 = fmaf(xa[w], yb[w], s01);
                    s10 = fmaf(xb[w], ya[w], s10);
                    s11 = fmaf(xb[w], yb[w], s11);
                }
            }
            far[i][0] = s00; far[i][1] = s01; far[i][2] = s10; far[i][3] = s11;
        }
    }
    float* A = a.weights + ((int64_t)blockIdx.x * H + head) * TC * TC;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        if (pt[i] >= 0) A[pt[i] * TC + psrc[i]] = pair[i];
        if (i == 1 && group >= 2) continue;
        float* at = A + (tb[i] * BT + ti) * TC + sb[i] * BT + si;
        *reinterpret_cast<float2*>(at) = make_float2(far[i][0], far[i][1]);
        *reinterpret_cast<float2*>(at + TC) = make_float2(far[i][2], far[i][3]);
    }
    own += __shfl_xor_sync(0xffffffffu, own, 1);
    own += __shfl_xor_sync(0xffffffffu, own, 2);
    if ((tid & 3) == 0) A[(tid >> 2) * TC + (tid >> 2)] = own;
    // (entries above the diagonal are never read)
}

// dS of one chunk and head: a tile of 64 key channels by 64 value columns; grid (slots, H, tiles),
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

// The read-outs of one chunk and head, 64 value columns; grid (slots, H, ceil(V / 64)), 128 threads:
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

template <typename T>
static cudaError_t launch_chunks(const ChannelArgs& a, int n_tokens, cudaStream_t stream) {
    const int slots = n_tokens / TC + a.n_rows + 1;
    const int nt = (a.N + 63) / 64, vt = (a.V + 63) / 64;
    const size_t smem = (size_t)W_FLOATS * sizeof(float);
    static bool ready = false;
    if (!ready) {
        cudaError_t e = cudaFuncSetAttribute(channel_weights_kernel<T>,
                                             cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
        ready = true;
    }
    cudaError_t e = sllm_launch_pdl(channel_weights_kernel<T>, dim3(slots, a.H), dim3(256), smem,
                                    stream, a);
    if (e != cudaSuccess) return e;
    e = sllm_launch_pdl(channel_state_kernel<T>, dim3(slots, a.H, nt * vt), dim3(128), 0, stream, a, nt);
    if (e != cudaSuccess) return e;
    const int64_t size = (int64_t)a.V * a.N;
    if ((a.N & 3) == 0)
        e = sllm_launch_pdl(channel_pass_kernel<4>, dim3((unsigned)((size / 4 + 255) / 256), a.H, a.n_rows),
                            dim3(256), 0, stream, a);
    else
        e = sllm_launch_pdl(channel_pass_kernel<1>, dim3((unsigned)((size + 255) / 256), a.H, a.n_rows),
                            dim3(256), 0, stream, a);
    if (e != cudaSuccess) return e;
    return sllm_launch_pdl(channel_out_kernel<T>, dim3(slots, a.H, vt), dim3(128), 0, stream, a);
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
    ChannelArgs a = {q, ldq, k, ldk, v, ldv, log_a, u, state, row_start, row_slot, out, scale,
                     H, N, V, vec4, 0x7fffffff, n_rows, dS, decay, weights};
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
