// A linear recurrence with one decay and one input weight per head and token: the state is a
// matrix S [N, V] per head and request, carried in 32-bit from token to token,
//
//     S  <-  a S + b k v^T,      o = scale * S^T q + skip * v        (0 <= a <= 1, b >= 0)
//
// with k, q of size N (head h of H reads group h / (H / G)), v of size V, a = exp(log_a).  A
// state-space layer (SSD) is this with k = B, q = C, a = exp(-rate dt), b = dt and a skip; a
// matrix memory with exponential gates is this with stabilised gates and a NORMALISER n <- a n +
// b k, which is one more column of S whose value is always 1 (`ones`): its read-out q . n goes to
// an array of its own.  Decays that are constants of the heads (lightning attention) are read from
// one array for all tokens (ld_gates 0), with b = 1 (b null); q, k and v may come ahead of a silu,
// which the first kernel then applies while it reads them.  The state is stored [slots, H, V (+ 1),
// N].
//
// gated_scan_kernel (any sizes, both dtypes, all arithmetic 32-bit): columns of S are
// independent.  LPC lanes share a column (EPL elements each, in quads), a CTA of 8 warps takes
// 8 * 32 / LPC columns of one (row, head) and walks the row's tokens in order, a chunk of them
// staged in shared memory at a time.  It serves decoding (one token), short portions, the 32-bit
// path and sizes that the chunk kernels below do not take.
//
// Long portions in bfloat16: chunks of TC = 64 tokens in parallel on the tensor cores.  With L_t
// the sum of log_a up to token t of a chunk and S0 the state at its start,
//
//     chunk_state   dS   = sum_s e^{L_last - L_s} b_s k_s v_s^T                 (every chunk at once)
//     chunk_pass    S0 of the next chunk = e^{L_last} S0 + dS                   (elementwise)
//     chunk_out     o_t  = e^{L_t} S0^T q_t + sum_{s <= t} e^{L_t - L_s} b_s (k_s . q_t) v_s
//
// Every exponent is at most 0.  k, q and v are bfloat16 already; what is 32-bit in these products
// (the weighted values, the weights of the second sum, the state S0) is split into three
// bfloat16 parts that hold all of its 24 bits, so that the products are those of the 32-bit
// numbers, accumulated in 32-bit.  The contractions are small (64 x 64 x N); what takes the time
// is the state's way through memory, so they run as mma.sync from shared memory, without the
// set-up of a TMEM accumulator.
//
// Chunks have slots (scan_chunks.cuh), so a launch over slots finds its chunk on the
// device and nothing is read on the host.  Rows of fewer than `min_chunked` tokens are the first
// kernel's, the others the chunk kernels'.
#include "scan_chunks.cuh"

namespace sllm {

struct ScanArgs {
    const void* q; int64_t ldq;          // [tokens, >= G * N]
    const void* k; int64_t ldk;          // [tokens, >= G * N]
    const void* v; int64_t ldv;          // [tokens, >= H * V]
    const float* log_a; const float* b;  // [tokens, H]; b null: 1
    int64_t ld_gates;                    // H, or 0: log_a is [H] for all tokens
    float* state;                        // [slots, H, VX, N], VX = V + ones
    const int* row_start; const int* row_slot;
    float* out;                          // [tokens, H * V]
    float* ones_out;                     // [tokens, H] or null
    const float* skip;                   // [H] or null
    float scale;
    int H, G, N, V, VX;
    int vec4;                            // rows of q and k allow reads of four elements
    int silu;                            // token-by-token kernel: q, k and v pass a silu
    int min_chunked;                     // rows of at least so many tokens are the chunk kernels'
    // chunk kernels only
    float* dS;                           // [slots of chunks, H, VX, N]
    float* decay;                        // [slots of chunks, H]: L of the chunk's last token
    int n_rows;
};

__device__ __forceinline__ float silu_if(float z, int on) { return on ? z / (1.0f + expf(-z)) : z; }
__device__ __forceinline__ float4 silu_if(float4 z, int on) {
    return on ? make_float4(silu_if(z.x, 1), silu_if(z.y, 1), silu_if(z.z, 1), silu_if(z.w, 1)) : z;
}

// ------------------------------------------------------------------------ token by token

template <typename T, int LPC, int EPL>
__global__ void __launch_bounds__(256) gated_scan_kernel(const ScanArgs a, int tokens_staged) {
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
    const int col = col0 + warp * (32 / LPC) + lane / LPC;
    const bool live = col < a.VX, is_ones = col >= a.V;
    const int N = a.N, V = a.V, H = a.H;
    const int g = head / (H / a.G);
    const T* q = reinterpret_cast<const T*>(a.q) + (int64_t)g * N;
    const T* k = reinterpret_cast<const T*>(a.k) + (int64_t)g * N;
    const T* v = reinterpret_cast<const T*>(a.v) + (int64_t)head * V;
    const float skip = a.skip ? a.skip[head] : 0.f;
    float* st = a.state + (((int64_t)a.row_slot[r] * H + head) * a.VX + (live ? col : 0)) * N;
    const bool quads = (N & 3) == 0;
    float S[EPL];
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
    }
    // decoding: nothing is staged (with a silu it is: every column's lanes would form it again)
    if (n_new == 1 && quads && a.vec4 && !a.silu) {
        const int64_t n = t0;
        const float decay = expf(a.log_a[n * a.ld_gates + head]);
        const float value = !is_ones ? to_float(v[n * a.ldv + col]) : 1.f;
        const float bv = a.b ? a.b[n * H + head] * value : value;
        float acc = 0.f;
#pragma unroll
        for (int i = 0; i < QPL; ++i) {
            const int e = (i * LPC + sub) * 4;
            if (e < N) {
                const float4 kk = load4(k + n * a.ldk + e), qq = load4(q + n * a.ldq + e);
                float4 x;
                x.x = fmaf(decay, S[4 * i], bv * kk.x);
                x.y = fmaf(decay, S[4 * i + 1], bv * kk.y);
                x.z = fmaf(decay, S[4 * i + 2], bv * kk.z);
                x.w = fmaf(decay, S[4 * i + 3], bv * kk.w);
                acc = fmaf(x.x, qq.x, fmaf(x.y, qq.y, fmaf(x.z, qq.z, fmaf(x.w, qq.w, acc))));
                if (live) *reinterpret_cast<float4*>(st + e) = x;
            }
        }
#pragma unroll
        for (int o = LPC / 2; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
        if (sub == 0 && live) {
            if (is_ones) a.ones_out[n * H + head] = acc * a.scale;
            else a.out[n * H * V + (int64_t)head * V + col] = fmaf(skip, value, acc * a.scale);
        }
        return;
    }
    const int NP = (N + 3) / 4 * 4;            // staged rows, padded with zeros
    float* ks = sm;                            // [tokens_staged][NP]
    float* qs = ks + tokens_staged * NP;       // [tokens_staged][NP]
    float* vs = qs + tokens_staged * NP;       // [tokens_staged][COLS]
    float* as = vs + tokens_staged * COLS;     // [tokens_staged]
    float* bs = as + tokens_staged;            // [tokens_staged]
    for (int c0 = 0; c0 < n_new; c0 += tokens_staged) {
        const int nt = min(tokens_staged, n_new - c0);
        if (c0) __syncthreads();               // the previous chunk is no longer read
        if (quads && a.vec4) {                 // four elements of a row at a time
            const int per = N / 4;
#pragma unroll 4
            for (int i = tid; i < nt * per; i += 256) {
                const int t = i / per, e = (i - t * per) * 4;
                const int64_t n = t0 + c0 + t;
                *reinterpret_cast<float4*>(ks + t * NP + e) = silu_if(load4(k + n * a.ldk + e), a.silu);
                *reinterpret_cast<float4*>(qs + t * NP + e) = silu_if(load4(q + n * a.ldq + e), a.silu);
            }
        } else {
            for (int i = tid; i < nt * NP; i += 256) {
                const int t = i / NP, e = i - t * NP;
                const int64_t n = t0 + c0 + t;
                ks[i] = e < N ? silu_if(to_float(k[n * a.ldk + e]), a.silu) : 0.f;
                qs[i] = e < N ? silu_if(to_float(q[n * a.ldq + e]), a.silu) : 0.f;
            }
        }
        for (int i = tid; i < nt * COLS; i += 256) {
            const int t = i / COLS, j = col0 + i - t * COLS;
            vs[i] = j < V ? silu_if(to_float(v[(int64_t)(t0 + c0 + t) * a.ldv + j]), a.silu) : 1.f;
        }
        for (int t = tid; t < nt; t += 256) {
            as[t] = expf(a.log_a[(int64_t)(t0 + c0 + t) * a.ld_gates + head]);
            bs[t] = a.b ? a.b[(int64_t)(t0 + c0 + t) * H + head] : 1.f;
        }
        __syncthreads();
        for (int t = 0; t < nt; ++t) {
            const float decay = as[t], value = vs[t * COLS + col - col0], bv = bs[t] * value;
            float part[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int i = 0; i < QPL; ++i) {
                const int e = (i * LPC + sub) * 4;
                if (e < NP) {
                    const float4 kk = *reinterpret_cast<const float4*>(ks + t * NP + e);
                    const float4 qq = *reinterpret_cast<const float4*>(qs + t * NP + e);
                    S[4 * i] = fmaf(decay, S[4 * i], bv * kk.x);
                    S[4 * i + 1] = fmaf(decay, S[4 * i + 1], bv * kk.y);
                    S[4 * i + 2] = fmaf(decay, S[4 * i + 2], bv * kk.z);
                    S[4 * i + 3] = fmaf(decay, S[4 * i + 3], bv * kk.w);
                    part[0] = fmaf(S[4 * i], qq.x, part[0]);
                    part[1] = fmaf(S[4 * i + 1], qq.y, part[1]);
                    part[2] = fmaf(S[4 * i + 2], qq.z, part[2]);
                    part[3] = fmaf(S[4 * i + 3], qq.w, part[3]);
                }
            }
            float acc = (part[0] + part[1]) + (part[2] + part[3]);
#pragma unroll
            for (int o = LPC / 2; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
            if (sub == 0 && live) {
                const int64_t n = t0 + c0 + t;
                if (is_ones) a.ones_out[n * H + head] = acc * a.scale;
                else a.out[n * H * V + (int64_t)head * V + col] = fmaf(skip, value, acc * a.scale);
            }
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

constexpr int VB = 64;          // columns of S per CTA (and the column of ones beside the last)
constexpr int VT = VB + 8;      // columns staged
constexpr int CHUNK_MAX_N = 256;
// Inclusive sums of log_a over the chunk's tokens into Ls[TC], b into bs[TC] (zero beyond the
// chunk's tokens), by the CTA's first warp.
__device__ __forceinline__ void chunk_gates(const ScanArgs& a, int64_t n0, int nt, int head,
                                            float* Ls, float* bs) {
    if (threadIdx.x >= 32) return;
    const int lane = threadIdx.x;
    const int64_t at = (n0 + 2 * lane) * a.ld_gates + head;
    const float x0 = 2 * lane < nt ? a.log_a[at] : 0.f;
    const float x1 = 2 * lane + 1 < nt ? a.log_a[at + a.ld_gates] : 0.f;
    const float* b = a.b ? a.b + (n0 + 2 * lane) * a.H + head : nullptr;
    bs[2 * lane] = 2 * lane < nt ? (b ? b[0] : 1.f) : 0.f;
    bs[2 * lane + 1] = 2 * lane + 1 < nt ? (b ? b[a.H] : 1.f) : 0.f;
    float sum = x0 + x1;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const float p = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += p;
    }
    float before = __shfl_up_sync(0xffffffffu, sum, 1);
    if (lane == 0) before = 0.f;
    Ls[2 * lane] = before + x0;
    Ls[2 * lane + 1] = before + x0 + x1;
}

// TC rows of N bfloat16 (N % 8 == 0, 16-byte aligned) into shared memory, row stride ld; rows from
// nt on are zero.
__device__ __forceinline__ void stage_rows(bf16* dst, int ld, const bf16* src, int64_t lds, int nt,
                                           int N) {
    const int units = N / 8, dt = blockDim.x / units, du = blockDim.x - dt * units;
    int t = threadIdx.x / units, u = threadIdx.x - t * units;
#pragma unroll 4
    for (; t < TC;) {
        uint4 x = make_uint4(0u, 0u, 0u, 0u);
        if (t < nt) x = *reinterpret_cast<const uint4*>(src + (int64_t)t * lds + u * 8);
        *reinterpret_cast<uint4*>(dst + t * ld + u * 8) = x;
        t += dt;
        u += du;
        if (u >= units) { u -= units; ++t; }
    }
}

// dS of one chunk and head, columns [v0, v0 + cols).  256 threads: the 16-row tiles of S's columns
// (m) against N (n), every warp an eighth of N's 8-wide tiles; the sum runs over the tokens.
__global__ void __launch_bounds__(256) chunk_state_kernel(const ScanArgs a) {
    extern __shared__ __align__(16) unsigned char raw[];
    __shared__ float Ls[TC], bs[TC], ws[TC];
    pdl_wait();
    pdl_trigger();
    int row, t0, c0, n_new;
    if (!find_chunk(a.row_start, a.n_rows, a.min_chunked, blockIdx.x, row, t0, c0, n_new)) return;
    const int head = blockIdx.y, v0 = blockIdx.z * VB;
    const int N = a.N, V = a.V, H = a.H;
    const int nt = min(TC, n_new - c0);
    const int64_t n0 = t0 + c0;
    const bool last_block = blockIdx.z == gridDim.z - 1;
    const int cols = last_block ? a.VX - v0 : VB;          // with the column of ones
    const int ldk = N + 8;
    constexpr int LDV = 80 + 8;                            // five tiles of 16 columns, padded
    bf16* ks = reinterpret_cast<bf16*>(raw);               // [TC][ldk]
    bf16* vs = ks + TC * ldk;                              // [PARTS][TC][LDV]: weighted values
    const bf16* k = reinterpret_cast<const bf16*>(a.k) + n0 * a.ldk + (int64_t)(head / (H / a.G)) * N;
    const bf16* v = reinterpret_cast<const bf16*>(a.v) + n0 * a.ldv + (int64_t)head * V;
    chunk_gates(a, n0, nt, head, Ls, bs);
    stage_rows(ks, ldk, k, a.ldk, nt, N);
    __syncthreads();
    const float L_last = Ls[TC - 1];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    if (tid == 0 && blockIdx.z == 0) a.decay[(int64_t)blockIdx.x * H + head] = L_last;
    const int m_tiles = (cols + 15) / 16;
    if (tid < TC) ws[tid] = expf(L_last - Ls[tid]) * bs[tid];
    __syncthreads();
    for (int jp = lane; jp < m_tiles * 8; jp += 32) {      // pairs of columns (V is even)
        const int j = jp * 2, c = v0 + j;
#pragma unroll
        for (int i = 0; i < TC / 8; ++i) {
            const int t = warp + i * 8;
            float x = 0.f, y = 0.f;
            if (t < nt && j < cols) {
                const float w = ws[t];
                x = w;                                     // the column of ones, and nothing behind
                if (c < V) {
                    const __nv_bfloat162 h =
                        *reinterpret_cast<const __nv_bfloat162*>(v + (int64_t)t * a.ldv + c);
                    x = __low2float(h) * w;
                    y = __high2float(h) * w;
                }
            }
            uint32_t part[PARTS];
            split2(x, y, part);
#pragma unroll
            for (int p = 0; p < PARTS; ++p)
                *reinterpret_cast<uint32_t*>(vs + (p * TC + t) * LDV + j) = part[p];
        }
    }
    __syncthreads();
    float* dst = a.dS + (((int64_t)blockIdx.x * H + head) * a.VX + v0) * N;
    const int n_tiles = N / 8;
    // warps w and w + 4: four of the n tiles at a time, every other of the m tiles
    for (int nb = (warp & 3) * 4; nb < n_tiles; nb += 16) {
        const bool wide = nb + 2 < n_tiles;                // (the number of n tiles is even)
        uint32_t bfrag[TC / 16][8];      // per 16 tokens: tiles nb .. nb + 3
#pragma unroll
        for (int kt = 0; kt < TC / 16; ++kt) {
            const bf16* at = ks + (kt * 16 + (lane & 15)) * ldk + nb * 8 + (lane >> 4) * 8;
            ldsm4_t(bfrag[kt], smem_addr(at));
            if (wide) ldsm4_t(bfrag[kt] + 4, smem_addr(at + 16));
        }
        for (int mt = warp >> 2; mt < m_tiles; mt += 2) {
            float acc[4][4];
#pragma unroll
            for (int u = 0; u < 4; ++u) acc[u][0] = acc[u][1] = acc[u][2] = acc[u][3] = 0.f;
#pragma unroll
            for (int p = PARTS - 1; p >= 0; --p)           // small parts first
#pragma unroll
                for (int kt = 0; kt < TC / 16; ++kt) {
                    // A[m = column][k = token] from [token][column]: transposed 8 x 8 blocks in the
                    // order (m 0-7, k 0-7), (m 8-15, k 0-7), (m 0-7, k 8-15), (m 8-15, k 8-15)
                    uint32_t af[4];
                    const int blk = lane >> 3;
                    ldsm4_t(af, smem_addr(vs + (p * TC + kt * 16 + (blk >> 1) * 8 + (lane & 7)) * LDV +
                                          mt * 16 + (blk & 1) * 8));
                    mma_bf16(acc[0], af, bfrag[kt]);
                    mma_bf16(acc[1], af, bfrag[kt] + 2);
                    if (wide) {
                        mma_bf16(acc[2], af, bfrag[kt] + 4);
                        mma_bf16(acc[3], af, bfrag[kt] + 6);
                    }
                }
            const int m = mt * 16 + (lane >> 2);
            float* d = dst + (int64_t)m * N + nb * 8 + (lane & 3) * 2;
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                if (nb + u >= n_tiles) break;
                if (m < cols) *reinterpret_cast<float2*>(d + u * 8) = make_float2(acc[u][0], acc[u][1]);
                if (m + 8 < cols)
                    *reinterpret_cast<float2*>(d + 8 * N + u * 8) = make_float2(acc[u][2], acc[u][3]);
            }
        }
    }
}

// The states at the chunks' starts, in place of the chunks' own dS, and the row's final state
// into its slot.  A thread per four elements; grid (ceil(VX N / 4 / 256), H, rows).
constexpr int PASS_AHEAD = 8;
__global__ void __launch_bounds__(256) chunk_pass_kernel(const ScanArgs a) {
    pdl_wait();
    pdl_trigger();
    const int r = blockIdx.z, head = blockIdx.y;
    const int t0 = a.row_start[r], n_new = a.row_start[r + 1] - t0;
    if (n_new < a.min_chunked) return;
    const int64_t size = (int64_t)a.VX * a.N;
    const int64_t e = ((int64_t)blockIdx.x * 256 + threadIdx.x) * 4;
    if (e >= size) return;
    const int n_chunks = (n_new + TC - 1) / TC;
    const int64_t slot0 = t0 / TC + r;
    float* d = a.dS + (slot0 * a.H + head) * size + e;
    const float* dec = a.decay + slot0 * a.H + head;
    const int64_t step = (int64_t)a.H * size;
    float4* home = reinterpret_cast<float4*>(a.state + ((int64_t)a.row_slot[r] * a.H + head) * size + e);
    float4 S = *home;
    for (int c0 = 0; c0 < n_chunks; c0 += PASS_AHEAD) {
        float4 x[PASS_AHEAD];
        float f[PASS_AHEAD];
#pragma unroll
        for (int i = 0; i < PASS_AHEAD; ++i)
            if (c0 + i < n_chunks) {
                x[i] = *reinterpret_cast<const float4*>(d + (c0 + i) * step);
                f[i] = dec[(int64_t)(c0 + i) * a.H];
            }
#pragma unroll
        for (int i = 0; i < PASS_AHEAD; ++i)
            if (c0 + i < n_chunks) {
                *reinterpret_cast<float4*>(d + (c0 + i) * step) = S;
                const float g = expf(f[i]);
                S.x = fmaf(g, S.x, x[i].x); S.y = fmaf(g, S.y, x[i].y);
                S.z = fmaf(g, S.z, x[i].z); S.w = fmaf(g, S.w, x[i].w);
            }
    }
    *home = S;
}

// The read-outs of one chunk and head, columns [v0, v0 + cols).  256 threads: warps w and w + 4 have
// the chunk's tokens 16 w .. 16 w + 15, and half of the columns' tiles each.  The keys, queries and
// state go through shared memory in slabs of KB elements of N.
constexpr int KB = 64, LDB = KB + 8;
constexpr int OT = (VT / 8 + 1) / 2;                       // column tiles of a warp
constexpr int OUT_LDV = VT + 16;
constexpr size_t OUT_SMEM = ((size_t)(2 * TC + PARTS * VT) * LDB + (size_t)TC * OUT_LDV) * sizeof(bf16);
__global__ void __launch_bounds__(256, 3) chunk_out_kernel(const ScanArgs a) {
    extern __shared__ __align__(16) unsigned char raw[];
    __shared__ float Ls[TC], bs[TC];
    pdl_wait();
    pdl_trigger();
    int row, t0, c0, n_new;
    if (!find_chunk(a.row_start, a.n_rows, a.min_chunked, blockIdx.x, row, t0, c0, n_new)) return;
    const int head = blockIdx.y, v0 = blockIdx.z * VB;
    const int N = a.N, V = a.V, H = a.H;
    const int nt = min(TC, n_new - c0);
    const int64_t n0 = t0 + c0;
    const bool last_block = blockIdx.z == gridDim.z - 1;
    const int cols = last_block ? a.VX - v0 : VB;
    const int n_tiles = (cols + 7) / 8;                    // up to VT / 8 = 9
    constexpr int LDV = OUT_LDV;
    bf16* ks = reinterpret_cast<bf16*>(raw);               // [TC][LDB]
    bf16* qs = ks + TC * LDB;                              // [TC][LDB]
    bf16* ss = qs + TC * LDB;                              // [PARTS][VT][LDB]: the state's columns
    bf16* vs = ss + PARTS * VT * LDB;                      // [TC][LDV]
    const int g = head / (H / a.G);
    const bf16* k = reinterpret_cast<const bf16*>(a.k) + n0 * a.ldk + (int64_t)g * N;
    const bf16* q = reinterpret_cast<const bf16*>(a.q) + n0 * a.ldq + (int64_t)g * N;
    const bf16* v = reinterpret_cast<const bf16*>(a.v) + n0 * a.ldv + (int64_t)head * V;
    const float* s0 = a.dS + (((int64_t)blockIdx.x * H + head) * a.VX + v0) * N;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    chunk_gates(a, n0, nt, head, Ls, bs);
    for (int i = tid; i < TC * n_tiles; i += 256) {        // eight values at a time
        const int t = i / n_tiles, j = (i - t * n_tiles) * 8;
        alignas(16) bf16 x[8];
        if (t < nt && v0 + j + 8 <= V) {
            *reinterpret_cast<uint4*>(x) = *reinterpret_cast<const uint4*>(v + (int64_t)t * a.ldv + v0 + j);
        } else {
#pragma unroll
            for (int w = 0; w < 8; ++w) {
                const int c = v0 + j + w;
                x[w] = t < nt && c < V ? v[(int64_t)t * a.ldv + c]
                                       : __float2bfloat16_rn(t < nt && c < a.VX ? 1.f : 0.f);
            }
        }
        *reinterpret_cast<uint4*>(vs + t * LDV + j) = *reinterpret_cast<const uint4*>(x);
    }
    const int m0 = (warp & 3) * 16, side = warp >> 2;
    const int first = side ? (n_tiles + 1) / 2 : 0;        // this warp's column tiles
    const int mine = side ? n_tiles / 2 : (n_tiles + 1) / 2;
    float o[OT][4];
#pragma unroll
    for (int j = 0; j < OT; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
    // k_s . q_t of this warp's tokens t and half of the tokens s: the groups of 16 with the
    // numbers side and side + 2
    float w[2][2][4];
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int u = 0; u < 4; ++u) w[i][0][u] = w[i][1][u] = 0.f;
    for (int kb = 0; kb < N; kb += KB) {
        const int width = min(KB, N - kb);
        if (kb) __syncthreads();                           // the previous slab is no longer read
        stage_rows(ks, LDB, k + kb, a.ldk, nt, width);
        stage_rows(qs, LDB, q + kb, a.ldq, nt, width);
        {   // S0's columns, split; zero columns up to a whole tile
            const int e = (tid & 15) * 4;
            if (e < width) {
#pragma unroll
                for (int i = 0; i < VT / 16 + 1; ++i) {
                    const int j = (tid >> 4) + i * 16;
                    if (j >= n_tiles * 8) break;
                    float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
                    if (j < cols) x = *reinterpret_cast<const float4*>(s0 + (int64_t)j * N + kb + e);
                    uint32_t lo[PARTS], hi[PARTS];
                    split2(x.x, x.y, lo);
                    split2(x.z, x.w, hi);
#pragma unroll
                    for (int p = 0; p < PARTS; ++p)
                        *reinterpret_cast<uint2*>(ss + (p * VT + j) * LDB + e) =
                            make_uint2(lo[p], hi[p]);
                }
            }
        }
        __syncthreads();
        for (int kt = 0; kt < width / 16; ++kt) {
            uint32_t af[4];
            ldsm4(af, smem_addr(qs + (m0 + (lane & 15)) * LDB + kt * 16 + (lane >> 4) * 8));
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int sg = (side + 2 * i) * 16;
                if (sg > m0) break;                       // later than this warp's tokens
                uint32_t bf[4];
                ldsm4(bf, smem_addr(ks + (sg + (lane >> 4) * 8 + (lane & 7)) * LDB + kt * 16 +
                                    ((lane >> 3) & 1) * 8));
                mma_bf16(w[i][0], af, bf);
                mma_bf16(w[i][1], af, bf + 2);
            }
#pragma unroll
            for (int p = PARTS - 1; p >= 0; --p)
#pragma unroll
                for (int j = 0; j < OT; j += 2) {          // two tiles a load
                    if (j >= mine) break;
                    uint32_t bf[4];
                    ldsm4(bf, smem_addr(ss + (p * VT + (first + j + (lane >> 4)) * 8 + (lane & 7)) * LDB +
                                        kt * 16 + ((lane >> 3) & 1) * 8));
                    mma_bf16(o[j], af, bf);
                    if (j + 1 < OT && j + 1 < mine) mma_bf16(o[j + 1], af, bf + 2);
                }
        }
    }
    const int ta = m0 + (lane >> 2), tb = ta + 8;          // this thread's two tokens
    const float La = Ls[ta], Lb = Ls[tb], ea = __expf(La), eb = __expf(Lb);
#pragma unroll
    for (int j = 0; j < OT; ++j) {
        o[j][0] *= ea; o[j][1] *= ea;
        o[j][2] *= eb; o[j][3] *= eb;
    }
    // the weights, split, into the state's place: [PARTS][TC][LDB]
    __syncthreads();
    bf16* ps = ss;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int sg = (side + 2 * i) * 16;
        if (sg > m0) break;
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            const int s = sg + h * 8 + (lane & 3) * 2;
            const float L0 = Ls[s], L1 = Ls[s + 1], b0 = bs[s], b1 = bs[s + 1];
            const float* x = w[i][h];
            uint32_t pa[PARTS], pb[PARTS];
            split2(s <= ta ? x[0] * __expf(La - L0) * b0 : 0.f,
                   s + 1 <= ta ? x[1] * __expf(La - L1) * b1 : 0.f, pa);
            split2(s <= tb ? x[2] * __expf(Lb - L0) * b0 : 0.f,
                   s + 1 <= tb ? x[3] * __expf(Lb - L1) * b1 : 0.f, pb);
#pragma unroll
            for (int p = 0; p < PARTS; ++p) {
                *reinterpret_cast<uint32_t*>(ps + (p * TC + ta) * LDB + s) = pa[p];
                *reinterpret_cast<uint32_t*>(ps + (p * TC + tb) * LDB + s) = pb[p];
            }
        }
    }
    __syncthreads();
#pragma unroll
    for (int kt = 0; kt < TC / 16; ++kt) {                 // tokens s of 16
        if (kt * 16 > m0) break;
        uint32_t af[PARTS][4];
#pragma unroll
        for (int p = 0; p < PARTS; ++p)
            ldsm4(af[p], smem_addr(ps + (p * TC + m0 + (lane & 15)) * LDB + kt * 16 + (lane >> 4) * 8));
#pragma unroll
        for (int j = 0; j < OT; ++j) {
            if (j >= mine) break;
            uint32_t bf[2];
            ldsm2_t(bf, smem_addr(vs + (kt * 16 + (lane & 15)) * LDV + (first + j) * 8));
#pragma unroll
            for (int p = PARTS - 1; p >= 0; --p) mma_bf16(o[j], af[p], bf);
        }
    }
    const float skip = a.skip ? a.skip[head] : 0.f;
#pragma unroll
    for (int j = 0; j < OT; ++j) {
        if (j >= mine) break;
        const int jc = (first + j) * 8 + (lane & 3) * 2, c = v0 + jc;
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int t = u ? tb : ta;
            if (t >= nt || c >= a.VX) continue;
            float x = o[j][2 * u] * a.scale, y = o[j][2 * u + 1] * a.scale;
            if (c >= V) {                                  // (V is even: the column of ones is x)
                a.ones_out[(n0 + t) * H + head] = x;
                continue;
            }
            if (skip != 0.f) {
                const __nv_bfloat162 h = *reinterpret_cast<const __nv_bfloat162*>(vs + t * LDV + jc);
                x = fmaf(skip, __low2float(h), x);
                y = fmaf(skip, __high2float(h), y);
            }
            *reinterpret_cast<float2*>(a.out + (n0 + t) * H * V + (int64_t)head * V + c) =
                make_float2(x, y);
        }
    }
}

}  // namespace sllm

using namespace sllm;

SLLM_EXPORT int sllm_gated_scan_chunk() { return TC; }

// Whether the chunk kernels take these sizes (bfloat16; the rows' alignment is checked at the call).
SLLM_EXPORT int sllm_gated_scan_chunks_fit(int N, int V) {
    return N % 16 == 0 && N <= CHUNK_MAX_N && V % 8 == 0;
}

// q, k: [n_tokens, >= G N], v: [n_tokens, >= H V] (dtype), log_a, b: float [n_tokens, H] (ld_gates H;
// ld_gates 0: log_a [H]; b may be null: 1); silu: q, k and v are taken through a silu (not with
// chunked); state:
// float [slots, H, V + ones, N]; out: float [n_tokens, H V]; ones_out: float [n_tokens, H] (ones
// only); skip: float [H] or null.  chunked: rows of at least min_chunked tokens take the chunk
// kernels, with the scratch dS float [n_tokens / 64 + n_rows + 1, H, V + ones, N] and decay float
// [the same, H]; else every row is walked token by token.  shortest / longest: bounds of the tokens
// a row brings.
SLLM_EXPORT int sllm_gated_scan(const void* q, int64_t ldq, const void* k, int64_t ldk,
                                const void* v, int64_t ldv, const float* log_a, const float* b,
                                int64_t ld_gates, int silu,
                                float* state, const int* row_start, const int* row_slot,
                                float* out, float* ones_out, const float* skip, float scale,
                                int n_tokens, int n_rows, int H, int G, int N, int V, int ones,
                                int chunked, int min_chunked, int shortest, int longest, float* dS,
                                float* decay, int dtype, cudaStream_t stream) {
    if (n_tokens <= 0 || n_rows <= 0) return 0;
    if (H < 1 || G < 1 || H % G || N < 1 || N > 1024 || V < 1 || ones < 0 || ones > 1 ||
        (ones && !ones_out) || ldq < (int64_t)G * N || ldk < (int64_t)G * N ||
        ldv < (int64_t)H * V || H > 65535 || n_rows > 65535 || dtype < 0 || dtype > 1 ||
        (ld_gates != 0 && ld_gates != H) || (silu && chunked))
        return (int)cudaErrorInvalidValue;
    const int vec4 = !((ldq | ldk | N) & 3) && !(((uintptr_t)q | (uintptr_t)k) & 15);
    ScanArgs a = {q, ldq, k, ldk, v, ldv, log_a, b, ld_gates, state, row_start, row_slot, out, ones_out,
                  skip, scale, H, G, N, V, V + ones, vec4, silu, 0x7fffffff, dS, decay, n_rows};
    if ((N & 3) == 0 && ((uintptr_t)state & 15)) return (int)cudaErrorInvalidValue;
    if (chunked) {
        if (dtype != 1 || !dS || !decay || min_chunked < 1 || !sllm_gated_scan_chunks_fit(N, V) ||
            ((ldq | ldk | ldv) & 7) ||
            (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)dS) & 15))
            return (int)cudaErrorInvalidValue;
        a.min_chunked = min_chunked;
        const int slots = n_tokens / TC + n_rows + 1;
        const int blocks_v = (V + VB - 1) / VB;
        const size_t smem_state = ((size_t)TC * (N + 8) + (size_t)PARTS * TC * 88) * sizeof(bf16);
        static bool ready = false;
        if (!ready) {
            cudaError_t e = cudaFuncSetAttribute(
                chunk_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024 - 1024);
            if (e == cudaSuccess)
                e = cudaFuncSetAttribute(chunk_out_kernel,
                                         cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         (int)OUT_SMEM);
            if (e != cudaSuccess) return (int)e;
            ready = true;
        }
        const int64_t quads = (int64_t)a.VX * N / 4;
        cudaError_t e = sllm_launch_pdl(chunk_state_kernel, dim3(slots, H, blocks_v), dim3(256),
                                        smem_state, stream, a);
        if (e != cudaSuccess) return (int)e;
        e = sllm_launch_pdl(chunk_pass_kernel, dim3((unsigned)((quads + 255) / 256), H, n_rows),
                            dim3(256), 0, stream, a);
        if (e != cudaSuccess) return (int)e;
        e = sllm_launch_pdl(chunk_out_kernel, dim3(slots, H, blocks_v), dim3(256), OUT_SMEM, stream,
                            a);
        if (e != cudaSuccess) return (int)e;
    }
    const int NP = (N + 3) / 4 * 4;
    int limit = longest > 0 ? longest : 32;
    if (chunked && limit > min_chunked - 1) limit = min_chunked - 1;
    if (limit < 1 || (chunked && shortest >= min_chunked)) return 0;   // nothing left
#define SLLM_SCAN(T, LPC, EPL)                                                                     \
    do {                                                                                           \
        constexpr int cols = 8 * 32 / LPC;                                                         \
        const int per = (2 * NP + cols + 2) * (int)sizeof(float);                                  \
        int staged = 47 * 1024 / per;                                                              \
        if (staged > 32) staged = 32;                                                              \
        if (staged > limit) staged = limit;                                                        \
        return (int)sllm_launch_pdl(gated_scan_kernel<T, LPC, EPL>,                                \
                                    dim3((a.VX + cols - 1) / cols, H, n_rows), dim3(256),          \
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
