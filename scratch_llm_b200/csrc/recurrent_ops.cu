// What stands around a linear recurrence in a recurrent mixer: the short causal convolution
// over time with its carried inputs, and the per-head norm and gate of the read-out.
//
//   conv:   y[t, c] = silu( bias[c] + sum_j taps[c, j] * x[t - (K - 1 - j), c] ),  j = 0 .. K-1
//           (the last tap multiplies the current token; before a sequence's start x is 0; the
//           bias is optional).
//           A request's last K - 1 inputs are carried in its state slot, state[slot, s, c] with
//           s = K - 2 the most recent, so that a row may bring any number of tokens per step.
//   update: the state after the row's tokens (a launch of its own: the convolution of a row's
//           first tokens reads the old state while its last tokens would overwrite it).
//   read-out: out[t, h, :] = o[t, h, :] / sqrt(mean(o[t, h, :]^2) + eps) * gain * silu(gate[t, h, :]),
//           optionally with o divided first by max(|den[t, h]|, floor[t, h]) + 1e-6; or, with the
//           gate ahead of the norm, y = o * silu(gate), each of several equal parts of y over
//           its own root mean square, times gain
//   gates of a scan with one decay and one input weight per head (gated_scan.cu)
//
// T is the dtype of matrix-product operands (float / bfloat16); taps, gains and the read-out
// o are 32-bit.  Tokens whose row is -1 are padding: their outputs are zero, nothing is carried.
#include "common.cuh"

namespace sllm {

constexpr int CONV_MAX_TAPS = 16;

// sigmoid(z): exact rounding steps on the 32-bit path; where the result is rounded to bfloat16 the
// hardware's exponential and division (relative error around 1e-6).
template <typename T> __device__ __forceinline__ float sigmoid_of(float z) {
    if (sizeof(T) == 4) return 1.0f / (1.0f + expf(-z));
    return __fdividef(1.0f, 1.0f + __expf(-z));
}

// V consecutive values (4: 16 or 8 bytes at a time, suitably aligned; 1: one by one).
template <int V> __device__ __forceinline__ void load_few(const float* p, float* v) {
    if (V == 4) {
        const float4 r = *reinterpret_cast<const float4*>(p);
        v[0] = r.x; v[V - 3] = r.y; v[V - 2] = r.z; v[V - 1] = r.w;
    } else {
        v[0] = p[0];
    }
}
template <int V> __device__ __forceinline__ void load_few(const __nv_bfloat16* p, float* v) {
    if (V == 4) {
        const uint2 r = *reinterpret_cast<const uint2*>(p);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&r);
        v[0] = __low2float(h[0]); v[V - 3] = __high2float(h[0]);
        v[V - 2] = __low2float(h[1]); v[V - 1] = __high2float(h[1]);
    } else {
        v[0] = __bfloat162float(p[0]);
    }
}
template <int V> __device__ __forceinline__ void store_few(float* p, const float* v) {
    if (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[V - 3], v[V - 2], v[V - 1]);
    else p[0] = v[0];
}
template <int V> __device__ __forceinline__ void store_few(__nv_bfloat16* p, const float* v) {
    if (V == 4) {
        uint2 r;
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&r);
        h[0] = __floats2bfloat162_rn(v[0], v[V - 3]);
        h[1] = __floats2bfloat162_rn(v[V - 2], v[V - 1]);
        *reinterpret_cast<uint2*>(p) = r;
    } else {
        p[0] = __float2bfloat16_rn(v[0]);
    }
}

// x: [n_tokens, ldx], the convolved channels are its first C columns.  out: [n_tokens, C].
template <typename T>
__global__ void conv_silu_kernel(const T* __restrict__ x, int64_t ldx,
                                 const float* __restrict__ taps, const float* __restrict__ bias,
                                 int K, const T* __restrict__ state,
                                 const int* __restrict__ token_row,
                                 const int* __restrict__ row_start,
                                 const int* __restrict__ row_slot, T* __restrict__ out, int C,
                                 int64_t n_tokens) {
    pdl_wait();
    pdl_trigger();
    const int64_t total = n_tokens * C;
    for (int64_t idx = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; idx < total;
         idx += (int64_t)gridDim.x * blockDim.x) {
        const int64_t n = idx / C;
        const int c = (int)(idx - n * C);
        const int r = token_row[n];
        if (r < 0) {
            out[idx] = from_float<T>(0.f);
            continue;
        }
        const int i = (int)(n - row_start[r]);           // index of the token within its row
        const T* st = state + (int64_t)row_slot[r] * (K - 1) * C;
        float acc = bias ? bias[c] : 0.f;
        for (int j = 0; j < K; ++j) {
            const int back = K - 1 - j;                  // how many tokens before this one
            float v;
            if (back <= i) v = to_float(x[(n - back) * ldx + c]);
            else v = to_float(st[(int64_t)(i + j) * C + c]);   // i - back + (K - 1)
            acc = fmaf(taps[(int64_t)c * K + j], v, acc);
        }
        out[idx] = from_float<T>(acc * sigmoid_of<T>(acc));
    }
}

// The same for bfloat16 with 16-byte accesses: a thread takes 8 consecutive channels of a token
// (C, ldx multiples of 8; 16-byte bases).  The arithmetic and its order are the scalar kernel's.
// taps_t is the taps' transpose [K, C], so that a thread's 8 taps of one time step are 32
// consecutive bytes and a warp's are consecutive too.
__global__ void conv_silu_vec_kernel(const __nv_bfloat16* __restrict__ x, int64_t ldx,
                                     const float* __restrict__ taps_t,
                                     const float* __restrict__ bias, int K,
                                     const __nv_bfloat16* __restrict__ state,
                                     const int* __restrict__ token_row,
                                     const int* __restrict__ row_start,
                                     const int* __restrict__ row_slot,
                                     __nv_bfloat16* __restrict__ out, int C, int64_t n_tokens) {
    pdl_wait();
    pdl_trigger();
    typedef __nv_bfloat16 bf16;
    const int per_row = C / 8;
    const int64_t total = n_tokens * per_row;
    for (int64_t idx = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; idx < total;
         idx += (int64_t)gridDim.x * blockDim.x) {
        const int64_t n = idx / per_row;
        const int c = (int)(idx - n * per_row) * 8;
        const int r = token_row[n];
        uint4 packed = make_uint4(0u, 0u, 0u, 0u);
        if (r >= 0) {
            const int i = (int)(n - row_start[r]);
            const bf16* st = state + (int64_t)row_slot[r] * (K - 1) * C;
            float acc[8];
#pragma unroll
            for (int w = 0; w < 8; ++w) acc[w] = bias ? bias[c + w] : 0.f;
            for (int j = 0; j < K; ++j) {
                const int back = K - 1 - j;
                const bf16* src = back <= i ? x + (n - back) * ldx + c : st + (int64_t)(i + j) * C + c;
                const uint4 raw = *reinterpret_cast<const uint4*>(src);
                const bf16* e = reinterpret_cast<const bf16*>(&raw);
                const float4 ta = *reinterpret_cast<const float4*>(taps_t + (int64_t)j * C + c);
                const float4 tb = *reinterpret_cast<const float4*>(taps_t + (int64_t)j * C + c + 4);
                const float tp[8] = {ta.x, ta.y, ta.z, ta.w, tb.x, tb.y, tb.z, tb.w};
#pragma unroll
                for (int w = 0; w < 8; ++w) acc[w] = fmaf(tp[w], __bfloat162float(e[w]), acc[w]);
            }
            bf16* o = reinterpret_cast<bf16*>(&packed);
#pragma unroll
            for (int w = 0; w < 8; ++w) o[w] = __float2bfloat16_rn(acc[w] * sigmoid_of<bf16>(acc[w]));
        }
        *reinterpret_cast<uint4*>(out + n * C + c) = packed;
    }
}

// Long steps: a thread takes 8 consecutive channels of CONV_RUN consecutive tokens, so that the
// taps are read once for all of them and every input once (the last K - 1 inputs stay in registers;
// at the start of the run, and where another row starts within it, they are read).  The
// arithmetic and its order are the scalar kernel's.
constexpr int CONV_RUN = 8;
template <int K>
__global__ void __launch_bounds__(128)
conv_silu_run_kernel(const __nv_bfloat16* __restrict__ x, int64_t ldx,
                     const float* __restrict__ taps_t, const float* __restrict__ bias,
                     const __nv_bfloat16* __restrict__ state, const int* __restrict__ token_row,
                     const int* __restrict__ row_start, const int* __restrict__ row_slot,
                     __nv_bfloat16* __restrict__ out, int C, int n_tokens) {
    pdl_wait();
    pdl_trigger();
    typedef __nv_bfloat16 bf16;
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
    if (c >= C) return;
    float tp[K][8], b[8];
#pragma unroll
    for (int j = 0; j < K; ++j) {
        Vec<float>::load(taps_t + (int64_t)j * C + c, tp[j]);
        Vec<float>::load(taps_t + (int64_t)j * C + c + 4, tp[j] + 4);
    }
#pragma unroll
    for (int w = 0; w < 8; ++w) b[w] = bias ? bias[c + w] : 0.f;
    const int n0 = blockIdx.y * CONV_RUN;
    int rows[CONV_RUN];                  // -1: padding, or beyond the last token
    uint4 in[CONV_RUN];                  // every input of the run is requested at once
#pragma unroll
    for (int i = 0; i < CONV_RUN; ++i) {
        const bool there = n0 + i < n_tokens;
        rows[i] = there ? token_row[n0 + i] : -1;
        in[i] = there ? *reinterpret_cast<const uint4*>(x + (int64_t)(n0 + i) * ldx + c)
                      : make_uint4(0u, 0u, 0u, 0u);
    }
    uint4 past[K > 1 ? K - 1 : 1];       // past[j]: the input K - 1 - j tokens before this one
    int row = -2;
#pragma unroll
    for (int k = 0; k < CONV_RUN; ++k) {
        const int n = n0 + k, r = rows[k];
        if (n >= n_tokens) break;
        uint4 packed = make_uint4(0u, 0u, 0u, 0u);
        if (r >= 0) {
            if (r != row) {
                const int i = n - row_start[r];
                const bf16* st = state + (int64_t)row_slot[r] * (K - 1) * C;
#pragma unroll
                for (int j = 0; j < K - 1; ++j) {
                    const int back = K - 1 - j;
                    past[j] = *reinterpret_cast<const uint4*>(
                        back <= i ? x + (int64_t)(n - back) * ldx + c : st + (int64_t)(i + j) * C + c);
                }
            }
            const uint4 now = in[k];
            float acc[8];
#pragma unroll
            for (int w = 0; w < 8; ++w) acc[w] = b[w];
#pragma unroll
            for (int j = 0; j < K; ++j) {
                const uint4 raw = j < K - 1 ? past[j] : now;
                const bf16* e = reinterpret_cast<const bf16*>(&raw);
#pragma unroll
                for (int w = 0; w < 8; ++w) acc[w] = fmaf(tp[j][w], __bfloat162float(e[w]), acc[w]);
            }
            bf16* o = reinterpret_cast<bf16*>(&packed);
#pragma unroll
            for (int w = 0; w < 8; ++w) o[w] = __float2bfloat16_rn(acc[w] * sigmoid_of<bf16>(acc[w]));
#pragma unroll
            for (int j = 0; j + 1 < K - 1; ++j) past[j] = past[j + 1];
            if (K > 1) past[K > 1 ? K - 2 : 0] = now;
        }
        row = r;
        *reinterpret_cast<uint4*>(out + (int64_t)n * C + c) = packed;
    }
}

// state[slot, s, c] for s = 0 .. K-2 becomes entry n_new + s of (old state, the row's new inputs).
// grid (ceil(C / 256), rows); rows without tokens are left alone.
template <typename T>
__global__ void conv_state_update_kernel(const T* __restrict__ x, int64_t ldx, int K,
                                         T* __restrict__ state, const int* __restrict__ row_start,
                                         const int* __restrict__ row_slot, int C) {
    pdl_wait();
    pdl_trigger();
    const int r = blockIdx.y;
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    const int t0 = row_start[r], n_new = row_start[r + 1] - t0;
    if (c >= C || n_new <= 0) return;
    T* st = state + (int64_t)row_slot[r] * (K - 1) * C;
    // ascending s reads old entries n_new + s > s only: in place is safe
    for (int s = 0; s < K - 1; ++s) {
        const int src = n_new + s;
        st[(int64_t)s * C + c] = src < K - 1 ? st[(int64_t)src * C + c]
                                             : x[(int64_t)(t0 + src - (K - 1)) * ldx + c];
    }
}

// grid (tokens, ceil(H / 4)); one warp per (token, head), or with WIDE (long heads) grid (tokens,
// H) and all four warps on one head.  o: [n_tokens, H * V] float;
// gate: rows ldg apart; out: rows ldo apart (a column slice of a wider buffer, or H * V).  gain has V entries (every head the same) or,
// with gain_per_head, H * V.  gate_act: 0 = silu(gate), 1 = sigmoid(gate).  den / floor (may be
// null): [n_tokens, H]; a head's o is first divided by max(|den|, floor) + 1e-6.
constexpr float DIVISOR_FLOOR = 1e-6f;
template <typename T, bool WIDE>
__global__ void __launch_bounds__(128)
head_norm_gate_kernel(const float* __restrict__ o, const T* __restrict__ gate, int64_t ldg,
                      const float* __restrict__ gain, float eps, const float* __restrict__ den,
                      const float* __restrict__ floor, T* __restrict__ out, int64_t ldo, int H,
                      int V, int gain_per_head, int gate_act) {
    pdl_wait();
    pdl_trigger();
    __shared__ float scratch[33];
    const int64_t n = blockIdx.x;
    const int head = WIDE ? blockIdx.y : blockIdx.y * 4 + (threadIdx.x >> 5);
    const int lane = WIDE ? threadIdx.x : threadIdx.x & 31;
    constexpr int lanes = WIDE ? 128 : 32;
    if (head >= H) return;                             // (never with WIDE)
    const float* src = o + (n * H + head) * V;
    float by = 1.f;
    if (den) by = 1.0f / (fmaxf(fabsf(den[n * H + head]), floor[n * H + head]) + DIVISOR_FLOOR);
    float ss = 0.f;
    for (int j = lane; j < V; j += lanes) {
        const float v = src[j] * by;
        ss += v * v;
    }
    ss = WIDE ? block_sum(ss, scratch) : warp_sum(ss);
    const float inv = by / sqrtf(ss / (float)V + eps);
    const T* g = gate + n * ldg + (int64_t)head * V;
    const float* gn = gain + (gain_per_head ? (int64_t)head * V : 0);
    T* dst = out + n * ldo + (int64_t)head * V;
    for (int j = lane; j < V; j += lanes) {
        const float z = to_float(g[j]);
        const float sig = sigmoid_of<T>(z);
        dst[j] = from_float<T>(src[j] * inv * gn[j] * (gate_act == 1 ? sig : z * sig));
    }
}

// The same four elements at a time, for heads of up to 128 entries in fours and no divisor: LANES
// lanes of a warp share a head (a lane has one quad), 128 threads a CTA.
template <typename T, int LANES>
__global__ void __launch_bounds__(128)
head_norm_gate_vec_kernel(const float* __restrict__ o, const T* __restrict__ gate, int64_t ldg,
                          const float* __restrict__ gain, float eps, T* __restrict__ out, int64_t ldo,
                          int H, int V, int gain_per_head, int gate_act, int64_t n_heads) {
    pdl_wait();
    pdl_trigger();
    const int64_t idx = (int64_t)blockIdx.x * (128 / LANES) + threadIdx.x / LANES;
    const int e = (threadIdx.x % LANES) * 4;
    const bool live = idx < n_heads && e < V;
    const int64_t n = live ? idx / H : 0;
    const int head = live ? (int)(idx - n * H) : 0;
    float v[4] = {0.f, 0.f, 0.f, 0.f}, z[4], gn[4];
    if (live) {
        load_few<4>(o + (n * H + head) * V + e, v);
        load_few<4>(gate + n * ldg + (int64_t)head * V + e, z);
        load_few<4>(gain + (gain_per_head ? (int64_t)head * V : 0) + e, gn);
    }
    float ss = (v[0] * v[0] + v[1] * v[1]) + (v[2] * v[2] + v[3] * v[3]);
#pragma unroll
    for (int k = LANES / 2; k > 0; k >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, k);
    if (!live) return;
    const float inv = 1.0f / sqrtf(ss / (float)V + eps);
#pragma unroll
    for (int k = 0; k < 4; ++k)
        v[k] = v[k] * inv * gn[k] * (gate_act == 1 ? 1.f : z[k]) * sigmoid_of<T>(z[k]);
    store_few<4>(out + n * ldo + (int64_t)head * V + e, v);
}

// Decays and removal rates of a delta-rule mixer whose decay comes through a low-rank pair of
// matrices.  pre: float32 [N, ldp] holds the removal rates' inputs in columns [0, C) and the
// low-rank hidden values in columns [C, C + R).  w2t: float32 [R, C] (the second matrix,
// transposed).  out: float32 [N, 2 C]:
//     out[n, c]     = exp(-decay_scale * sigmoid(w0[c] + sum_r w2t[r, c] * tanh(pre[n, C + r])))
//     out[n, C + c] = sigmoid(pre[n, c] + a_bias[c])
// All in 32-bit; the sum runs over r in ascending order for every token, whatever the batch.
// grid (ceil(C / 256), ceil(N / LOWRANK_TOKENS)); shared: LOWRANK_TOKENS * R floats.
constexpr int LOWRANK_TOKENS = 8;
__global__ void __launch_bounds__(256)
lowrank_decay_kernel(const float* __restrict__ pre, int64_t ldp, const float* __restrict__ w2t,
                     const float* __restrict__ w0, const float* __restrict__ a_bias,
                     float decay_scale, float* __restrict__ out, int N, int C, int R) {
    pdl_wait();
    pdl_trigger();
    extern __shared__ float th[];   // [LOWRANK_TOKENS][R]
    const int n0 = blockIdx.y * LOWRANK_TOKENS;
    const int nt = min(LOWRANK_TOKENS, N - n0);
    for (int i = threadIdx.x; i < LOWRANK_TOKENS * R; i += blockDim.x) {
        const int t = i / R, r = i - t * R;
        th[t * R + r] = t < nt ? tanhf(pre[(int64_t)(n0 + t) * ldp + C + r]) : 0.f;
    }
    __syncthreads();
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= C) return;
    float acc[LOWRANK_TOKENS];
#pragma unroll
    for (int t = 0; t < LOWRANK_TOKENS; ++t) acc[t] = 0.f;
    // (sixteen weights are requested at a time: the loop is bound by their latency, not by its
    // arithmetic; tokens beyond nt have zeros in shared memory)
    int r = 0;
    for (; r + 16 <= R; r += 16) {
        float w[16];
#pragma unroll
        for (int j = 0; j < 16; ++j) w[j] = w2t[(int64_t)(r + j) * C + c];
#pragma unroll
        for (int j = 0; j < 16; ++j)
#pragma unroll
            for (int t = 0; t < LOWRANK_TOKENS; ++t) acc[t] = fmaf(w[j], th[t * R + r + j], acc[t]);
    }
    for (; r < R; ++r) {
        const float w = w2t[(int64_t)r * C + c];
#pragma unroll
        for (int t = 0; t < LOWRANK_TOKENS; ++t) acc[t] = fmaf(w, th[t * R + r], acc[t]);
    }
    const float b0 = w0[c], ab = a_bias[c];
#pragma unroll
    for (int t = 0; t < LOWRANK_TOKENS; ++t) {
        if (t < nt) {
            const int64_t n = n0 + t;
            const float sg = 1.0f / (1.0f + expf(-(acc[t] + b0)));
            out[n * 2 * C + c] = expf(-decay_scale * sg);
            out[n * 2 * C + C + c] = 1.0f / (1.0f + expf(-(pre[n * ldp + c] + ab)));
        }
    }
}

// The second product of a low-rank pair, in 32-bit, with what follows it.  pre: float32 [N, ldp]
// holds the hidden values (the first product's output) in columns [col0, col0 + R); w2t: float32
// [R, C] (the second matrix, transposed); bias (may be null): float32 [C].
//     z[n, c] = bias[c] + sum_r w2t[r, c] * pre[n, col0 + r]
//     mode 0:  out = z
//     mode 1:  out = -exp(rate_log[c / per_rate]) * softplus(z)    (the logarithm of a decay
//              exp(-exp(A) softplus(z)) with one A per `per_rate` channels)
//     mode 2:  out = rate * log sigmoid(z)                         (of a decay sigmoid(z)^rate)
//     mode 3:  out = -exp(z)                                       (of a decay exp(-exp(z)))
// In modes 2 and 3 out is at least LOG_DECAY_FLOOR: beyond it a state is zero in 32-bit within a
// token, and sums of such logarithms keep their precision.  tanh_in: the hidden values pass a tanh.
// The sum runs over r in ascending order for every token, whatever the batch.  out: [N, C],
// float32 or bfloat16.  One launch serves up to two such products of the same `pre` (a mixer's
// decays and its gate): the first `blocks0` CTAs along x take the first job, the rest the second.
// grid (blocks of both jobs, ceil(N / TOKENS)); shared: TOKENS * max R floats (R up to a multiple of 4).
constexpr float LOG_DECAY_FLOOR = -88.f;
struct ExpandJob {
    int col0; const float* w2t; const float* bias; const float* rate_log; int per_rate; int mode;
    float rate; int tanh_in;
    void* out; int out_bf16; int C; int R;
};

// A CTA has TOKENS tokens and CH channels a thread (2: C even); a thread's next AHEAD rows of
// weights are in flight while it works on the ones before, the first ones already before the kernel
// waits for those ahead of it (nothing writes weights).
template <int TOKENS, int CH, int AHEAD>
__global__ void __launch_bounds__(256)
lowrank_expand_kernel(const float* __restrict__ pre, int64_t ldp, const ExpandJob j0,
                      const ExpandJob j1, int blocks0, int N) {
    extern __shared__ __align__(16) float th[];   // [TOKENS][RP], zeros from R on
    struct alignas(4 * CH) Weights { float x[CH]; };
    const bool second = (int)blockIdx.x >= blocks0;
    const ExpandJob& j = second ? j1 : j0;
    const int R = j.R, C = j.C, RP = (R + 3) / 4 * 4;
    const int n0 = blockIdx.y * TOKENS;
    const int nt = min(TOKENS, N - n0);
    const int c = (((int)blockIdx.x - (second ? blocks0 : 0)) * blockDim.x + threadIdx.x) * CH;
    const float* w2t = j.w2t + (c < C ? c : 0);
    const Weights none = {};
    Weights w[AHEAD];
#pragma unroll
    for (int k = 0; k < AHEAD; ++k)
        w[k] = k < R ? *reinterpret_cast<const Weights*>(w2t + (int64_t)k * C) : none;
    pdl_wait();
    pdl_trigger();
    for (int i = threadIdx.x; i < TOKENS * RP; i += blockDim.x) {
        const int t = i / RP, r = i - t * RP;
        const float h = t < nt && r < R ? pre[(int64_t)(n0 + t) * ldp + j.col0 + r] : 0.f;
        th[i] = j.tanh_in ? tanhf(h) : h;
    }
    __syncthreads();
    if (c >= C) return;
    float acc[TOKENS][CH];
#pragma unroll
    for (int t = 0; t < TOKENS; ++t)
#pragma unroll
        for (int h = 0; h < CH; ++h) acc[t][h] = 0.f;
    for (int r = 0; r < R; r += AHEAD) {
        Weights next[AHEAD];
#pragma unroll
        for (int k = 0; k < AHEAD; ++k)
            next[k] = r + AHEAD + k < R
                ? *reinterpret_cast<const Weights*>(w2t + (int64_t)(r + AHEAD + k) * C) : none;
#pragma unroll
        for (int k = 0; k < AHEAD; k += 4) {
            if (r + k >= R) break;
#pragma unroll
            for (int t = 0; t < TOKENS; ++t) {
                float x[4];
                *reinterpret_cast<float4*>(x) = *reinterpret_cast<const float4*>(th + t * RP + r + k);
#pragma unroll
                for (int u = 0; u < 4; ++u)
#pragma unroll
                    for (int h = 0; h < CH; ++h) acc[t][h] = fmaf(w[k + u].x[h], x[u], acc[t][h]);
            }
        }
#pragma unroll
        for (int k = 0; k < AHEAD; ++k) w[k] = next[k];
    }
    float b0[CH], rate[CH];
#pragma unroll
    for (int h = 0; h < CH; ++h) {
        b0[h] = j.bias ? j.bias[c + h] : 0.f;
        rate[h] = j.mode == 1 ? expf(j.rate_log[(c + h) / j.per_rate]) : 0.f;
    }
#pragma unroll
    for (int t = 0; t < TOKENS; ++t) {
        if (t >= nt) break;
#pragma unroll
        for (int h = 0; h < CH; ++h) {
            float z = acc[t][h] + b0[h];
            if (j.mode == 1) z = -rate[h] * (z > 20.f ? z : log1pf(expf(z)));
            else if (j.mode == 2)
                z = fmaxf(j.rate * (fminf(z, 0.f) - log1pf(expf(-fabsf(z)))), LOG_DECAY_FLOOR);
            else if (j.mode == 3) z = fmaxf(-expf(z), LOG_DECAY_FLOOR);
            acc[t][h] = z;
        }
        const int64_t at = (int64_t)(n0 + t) * C + c;
        if (j.out_bf16) {
#pragma unroll
            for (int h = 0; h < CH; ++h)
                reinterpret_cast<__nv_bfloat16*>(j.out)[at + h] = __float2bfloat16_rn(acc[t][h]);
        } else {
            Weights out;
#pragma unroll
            for (int h = 0; h < CH; ++h) out.x[h] = acc[t][h];
            *reinterpret_cast<Weights*>(reinterpret_cast<float*>(j.out) + at) = out;
        }
    }
}

// The gate ahead of the norm: y = o * act(gate), then each of `parts` equal parts of y over its
// own root mean square, times gain [W]; or (after) the norm of o first, then the gate: out = o over
// its part's root mean square, times gain, times act(gate).  gate_act: 0 = silu, 1 = sigmoid.  o: float [n_tokens, W]; one CTA per (token, part), a
// part of P = W / parts elements waits in shared memory between the two passes.  V: elements per
// access (4 where P and the rows allow 16-byte reads of o, else 1).
template <typename T, int V>
__global__ void __launch_bounds__(256)
gate_part_norm_kernel(const float* __restrict__ o, const T* __restrict__ gate, int64_t ldg,
                      const float* __restrict__ gain, float eps, T* __restrict__ out, int64_t ldo,
                      int W, int P, int gate_act, int after) {
    pdl_wait();
    pdl_trigger();
    extern __shared__ __align__(16) float gp_row[];     // [P]
    __shared__ float scratch[33];
    const int64_t n = blockIdx.x;
    const int at = blockIdx.y * P;
    float ss = 0.f;
    for (int i = threadIdx.x * V; i < P; i += blockDim.x * V) {
        float v[V], z[V];
        load_few<V>(o + n * W + at + i, v);
        if (!after) {
            load_few<V>(gate + n * ldg + at + i, z);
#pragma unroll
            for (int k = 0; k < V; ++k) v[k] *= (gate_act ? 1.f : z[k]) * sigmoid_of<T>(z[k]);
        }
#pragma unroll
        for (int k = 0; k < V; ++k) {
            ss = fmaf(v[k], v[k], ss);
            gp_row[i + k] = v[k];
        }
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)P + eps);
    for (int i = threadIdx.x * V; i < P; i += blockDim.x * V) {
        float v[V];
#pragma unroll
        for (int k = 0; k < V; ++k) v[k] = gp_row[i + k] * inv * gain[at + i + k];
        if (after) {
            float z[V];
            load_few<V>(gate + n * ldg + at + i, z);
#pragma unroll
            for (int k = 0; k < V; ++k) v[k] *= (gate_act ? 1.f : z[k]) * sigmoid_of<T>(z[k]);
        }
        store_few<V>(out + n * ldo + at + i, v);
    }
}

// Gates of a scan with one decay and one input weight per head (gated_scan.cu), from 32-bit
// projections.  A state-space layer: b = softplus(x + bias), log_a = -exp(A_log) * b; element
// by element.  pre: rows ldp apart, the first H columns.
__global__ void ssd_gates_kernel(const float* __restrict__ pre, int64_t ldp,
                                 const float* __restrict__ bias, const float* __restrict__ A_log,
                                 float* __restrict__ log_a, float* __restrict__ b, int n_tokens,
                                 int H) {
    pdl_wait();
    pdl_trigger();
    for (int64_t i = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; i < (int64_t)n_tokens * H;
         i += (int64_t)gridDim.x * blockDim.x) {
        const int64_t n = i / H;
        const int h = (int)(i - n * H);
        const float x = pre[n * ldp + h] + bias[h];
        const float step = x > 20.f ? x : log1pf(expf(x));
        b[i] = step;
        log_a[i] = -expf(A_log[h]) * step;
    }
}

// A matrix memory with exponential gates: pre holds the input gates' sums in columns [0, H), the
// forget gates' in [H, 2H).  i = cap tanh((x_i + b_i) / cap), f = log sigmoid(cap tanh((x_f +
// b_f) / cap)); a running maximum m (one per slot and head, carried in `running`) keeps the state
// in range: m_t = max(f + m_(t-1), i), log_a = f + m_(t-1) - m_t, b = exp(i - m_t), floor =
// exp(-m_t).  (log_a and i - m_t are at most 0.)
struct MemoryGates {
    const float* pre; int64_t ldp; const float* bi; const float* bf; float cap;
    float* running; const int* row_start; const int* row_slot;
    float* log_a; float* b; float* floor; int H;
};
__device__ __forceinline__ void memory_gate_inputs(const MemoryGates& a, int64_t n, int h, float& i,
                                                   float& f) {
    i = a.cap * tanhf((a.pre[n * a.ldp + h] + a.bi[h]) / a.cap);
    const float z = a.cap * tanhf((a.pre[n * a.ldp + a.H + h] + a.bf[h]) / a.cap);
    f = fminf(z, 0.f) - log1pf(expf(-fabsf(z)));
}
// Rows of one token each (and rows without tokens): a thread per (row, head).
__global__ void memory_gates_step_kernel(const MemoryGates a, int n_rows) {
    pdl_wait();
    pdl_trigger();
    const int idx = blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= n_rows * a.H) return;
    const int r = idx / a.H, h = idx - r * a.H;
    const int64_t n = a.row_start[r];
    if (a.row_start[r + 1] <= n) return;
    float i, f;
    memory_gate_inputs(a, n, h, i, f);
    float* m = a.running + (int64_t)a.row_slot[r] * a.H + h;
    const float before = *m, now = fmaxf(f + before, i);
    a.log_a[n * a.H + h] = f + before - now;
    a.b[n * a.H + h] = expf(i - now);
    a.floor[n * a.H + h] = expf(-now);
    *m = now;
}
// Rows of any length: a CTA per (head, row), 256 tokens at a time.  The running maximum is a scan
// over pairs (F, M): a token maps m to max(F + m, M) with (F, M) = (f, i), and two maps in a
// row are (F1 + F2, max(M1 + F2, M2)).
__global__ void __launch_bounds__(256) memory_gates_kernel(const MemoryGates a) {
    pdl_wait();
    pdl_trigger();
    __shared__ float wF[8], wM[8];
    const int h = blockIdx.x, r = blockIdx.y;
    const int t0 = a.row_start[r], n_new = a.row_start[r + 1] - t0;
    if (n_new <= 0) return;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    float* m = a.running + (int64_t)a.row_slot[r] * a.H + h;
    float carried = *m;
    for (int c0 = 0; c0 < n_new; c0 += 256) {
        const int t = c0 + tid;
        float i = -INFINITY, f = 0.f;          // (tokens beyond the row change nothing)
        if (t < n_new) memory_gate_inputs(a, t0 + t, h, i, f);
        float F = f, M = i;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float Fp = __shfl_up_sync(0xffffffffu, F, o), Mp = __shfl_up_sync(0xffffffffu, M, o);
            if (lane >= o) {
                M = fmaxf(Mp + F, M);
                F += Fp;
            }
        }
        __syncthreads();                       // the last round's sums are no longer read
        if (lane == 31) { wF[warp] = F; wM[warp] = M; }
        __syncthreads();
        float start = carried;                 // m ahead of this warp's tokens
        for (int w = 0; w < warp; ++w) start = fmaxf(wF[w] + start, wM[w]);
        const float Fp = __shfl_up_sync(0xffffffffu, F, 1), Mp = __shfl_up_sync(0xffffffffu, M, 1);
        const float before = lane == 0 ? start : fmaxf(Fp + start, Mp);
        if (t < n_new) {
            const float now = fmaxf(f + before, i);
            const int64_t at = (int64_t)(t0 + t) * a.H + h;
            a.log_a[at] = f + before - now;
            a.b[at] = expf(i - now);
            a.floor[at] = expf(-now);
        }
        for (int w = 0; w < 8; ++w) carried = fmaxf(wF[w] + carried, wM[w]);
    }
    if (tid == 0) *m = carried;
}

// A token shift in front of several projections: with h' the previous token's h (a row's first
// token: what the slot carries, zeros at a sequence's start), out[m, n, :] = h + (h' - h) * mu[m] for
// m = 0 .. M - 1.  The row's last h is left in the slot by whoever takes the row's first token, after
// the old one has been read.  h [n_tokens, d], mu [M, d], state [slots, d] (32-bit), out [M, n_tokens,
// d].  A thread takes V channels of SHIFT_RUN consecutive tokens.  Padding tokens (row -1) get zeros.
constexpr int SHIFT_RUN = 4;
template <typename T, int V>
__global__ void __launch_bounds__(128)
shift_mix_kernel(const T* __restrict__ h, int64_t ldh, const float* __restrict__ mu, int M,
                 float* __restrict__ state, const int* __restrict__ token_row,
                 const int* __restrict__ row_start, const int* __restrict__ row_slot,
                 T* __restrict__ out, int d, int n_tokens) {
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
    pdl_wait();
    pdl_trigger();
    if (c >= d) return;
    const int n0 = blockIdx.y * SHIFT_RUN;
    float now[SHIFT_RUN][V], before[SHIFT_RUN][V];
    int rows[SHIFT_RUN];
#pragma unroll
    for (int i = 0; i < SHIFT_RUN; ++i) {
        rows[i] = n0 + i < n_tokens ? token_row[n0 + i] : -1;
#pragma unroll
        for (int k = 0; k < V; ++k) now[i][k] = before[i][k] = 0.f;
        if (rows[i] >= 0) load_few<V>(h + (int64_t)(n0 + i) * ldh + c, now[i]);
    }
#pragma unroll
    for (int i = 0; i < SHIFT_RUN; ++i) {
        const int r = rows[i], n = n0 + i;
        if (r < 0) continue;
        if (n > row_start[r]) {
            if (i) {
#pragma unroll
                for (int k = 0; k < V; ++k) before[i][k] = now[i ? i - 1 : 0][k];
            } else {
                load_few<V>(h + (int64_t)(n - 1) * ldh + c, before[i]);
            }
        } else {
            float* mine = state + (int64_t)row_slot[r] * d + c;
            float last[V];
            load_few<V>(mine, before[i]);
            load_few<V>(h + (int64_t)(row_start[r + 1] - 1) * ldh + c, last);
            store_few<V>(mine, last);
        }
    }
    for (int m = 0; m < M; ++m) {
        float w[V];
        load_few<V>(mu + (int64_t)m * d + c, w);
#pragma unroll
        for (int i = 0; i < SHIFT_RUN; ++i) {
            if (n0 + i >= n_tokens) break;
            float x[V];
#pragma unroll
            for (int k = 0; k < V; ++k) x[k] = fmaf(before[i][k] - now[i][k], w[k], now[i][k]);
            store_few<V>(out + ((int64_t)m * n_tokens + n0 + i) * d + c, x);
        }
    }
}

// silu in place on the first C columns of x's rows.
template <typename T, int V>
__global__ void silu_columns_kernel(T* __restrict__ x, int64_t ldx, int C, int64_t n_items) {
    pdl_wait();
    pdl_trigger();
    const int per_row = C / V;
    for (int64_t i = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; i < n_items;
         i += (int64_t)gridDim.x * blockDim.x) {
        const int64_t n = i / per_row;
        T* p = x + n * ldx + (i - n * per_row) * V;
        float z[V];
        load_few<V>(p, z);
#pragma unroll
        for (int k = 0; k < V; ++k) z[k] *= sigmoid_of<T>(z[k]);
        store_few<V>(p, z);
    }
}

}  // namespace sllm

using namespace sllm;

// dtype: 0 = float32, 1 = bfloat16 (of x, state, out, gate).
// bias (may be null): [C].  taps_t (may be null): the transpose [K, C] of taps, which the kernel with 16-byte accesses reads.
SLLM_EXPORT int sllm_conv_silu(const void* x, int64_t ldx, const float* taps,
                               const float* taps_t, const float* bias, int K,
                               const void* state, const int* token_row, const int* row_start,
                               const int* row_slot, void* out, int C, int n_tokens, int dtype,
                               cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (C <= 0 || K < 1 || K > CONV_MAX_TAPS || ldx < C) return (int)cudaErrorInvalidValue;
    if (dtype == 1 && taps_t != nullptr && C % 8 == 0 && ldx % 8 == 0 &&
        !(((uintptr_t)x | (uintptr_t)state | (uintptr_t)out | (uintptr_t)taps_t) & 15)) {
        if (n_tokens >= 256 && K <= 4 && (n_tokens + CONV_RUN - 1) / CONV_RUN <= 65535) {
            dim3 grid((C / 8 + 127) / 128, (n_tokens + CONV_RUN - 1) / CONV_RUN);
            typedef __nv_bfloat16 bf16;
            auto run = K == 1 ? conv_silu_run_kernel<1> : K == 2 ? conv_silu_run_kernel<2>
                     : K == 3 ? conv_silu_run_kernel<3> : conv_silu_run_kernel<4>;
            return (int)sllm_launch_pdl(run, grid, dim3(128), 0, stream, (const bf16*)x, ldx, taps_t,
                                        bias, (const bf16*)state, token_row, row_start, row_slot,
                                        (bf16*)out, C, n_tokens);
        }
        int64_t vblocks = ((int64_t)n_tokens * (C / 8) + 255) / 256;
        if (vblocks > 148 * 32) vblocks = 148 * 32;
        conv_silu_vec_kernel<<<(int)vblocks, 256, 0, stream>>>(
            (const __nv_bfloat16*)x, ldx, taps_t, bias, K, (const __nv_bfloat16*)state, token_row,
            row_start, row_slot, (__nv_bfloat16*)out, C, n_tokens);
        SLLM_LAUNCH_CHECK();
        return 0;
    }
    int64_t blocks = ((int64_t)n_tokens * C + 255) / 256;
    if (blocks > 148 * 32) blocks = 148 * 32;
    if (dtype == 0)
        conv_silu_kernel<float><<<(int)blocks, 256, 0, stream>>>(
            (const float*)x, ldx, taps, bias, K, (const float*)state, token_row, row_start, row_slot,
            (float*)out, C, n_tokens);
    else if (dtype == 1)
        conv_silu_kernel<__nv_bfloat16><<<(int)blocks, 256, 0, stream>>>(
            (const __nv_bfloat16*)x, ldx, taps, bias, K, (const __nv_bfloat16*)state, token_row,
            row_start, row_slot, (__nv_bfloat16*)out, C, n_tokens);
    else
        return (int)cudaErrorInvalidValue;
    SLLM_LAUNCH_CHECK();
    return 0;
}

SLLM_EXPORT int sllm_conv_state_update(const void* x, int64_t ldx, int K, void* state,
                                       const int* row_start, const int* row_slot, int C,
                                       int n_rows, int dtype, cudaStream_t stream) {
    if (n_rows <= 0 || K <= 1) return 0;
    if (C <= 0 || K > CONV_MAX_TAPS || n_rows > 65535) return (int)cudaErrorInvalidValue;
    dim3 grid((C + 255) / 256, n_rows);
    if (dtype == 0)
        conv_state_update_kernel<float><<<grid, 256, 0, stream>>>(
            (const float*)x, ldx, K, (float*)state, row_start, row_slot, C);
    else if (dtype == 1)
        conv_state_update_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>(
            (const __nv_bfloat16*)x, ldx, K, (__nv_bfloat16*)state, row_start, row_slot, C);
    else
        return (int)cudaErrorInvalidValue;
    SLLM_LAUNCH_CHECK();
    return 0;
}

SLLM_EXPORT int sllm_head_norm_gate(const float* o, const void* gate, int64_t ldg,
                                    const float* gain, float eps, const float* den,
                                    const float* floor, void* out, int64_t ldo, int n_tokens, int H, int V, int gain_per_head, int gate_act,
                                    int dtype, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (H <= 0 || V <= 0 || gate_act < 0 || gate_act > 1 || ldo < (int64_t)H * V ||
        (den == nullptr) != (floor == nullptr))
        return (int)cudaErrorInvalidValue;
    const int wide = V >= 256 && (int64_t)n_tokens * H <= 1024;
    dim3 grid(n_tokens, wide ? H : (H + 3) / 4);
    if (H > 65535) return (int)cudaErrorInvalidValue;
    typedef __nv_bfloat16 bf16;
    if (!den && V % 4 == 0 && V <= 128 && ldg % 4 == 0 && ldo % 4 == 0 &&
        !(((uintptr_t)o | (uintptr_t)gate | (uintptr_t)gain | (uintptr_t)out) & 15)) {
        const int64_t heads = (int64_t)n_tokens * H;
        const int lanes = V <= 16 ? 4 : V <= 32 ? 8 : V <= 64 ? 16 : 32;
        const unsigned blocks = (unsigned)((heads + 128 / lanes - 1) / (128 / lanes));
#define SLLM_HNV(T, L)                                                                             \
    return (int)sllm_launch_pdl(head_norm_gate_vec_kernel<T, L>, dim3(blocks), dim3(128), 0, stream, \
                                o, (const T*)gate, ldg, gain, eps, (T*)out, ldo, H, V,             \
                                gain_per_head, gate_act, heads)
#define SLLM_HNV_T(T)                                                                              \
    do {                                                                                           \
        if (lanes == 4) SLLM_HNV(T, 4);                                                            \
        if (lanes == 8) SLLM_HNV(T, 8);                                                            \
        if (lanes == 16) SLLM_HNV(T, 16);                                                          \
        SLLM_HNV(T, 32);                                                                           \
    } while (0)
        if (dtype == 0) SLLM_HNV_T(float);
        if (dtype == 1) SLLM_HNV_T(bf16);
#undef SLLM_HNV_T
#undef SLLM_HNV
    }
#define SLLM_HNG(T, WIDE)                                                                          \
    head_norm_gate_kernel<T, WIDE><<<grid, 128, 0, stream>>>(o, (const T*)gate, ldg, gain, eps, den, \
                                                             floor, (T*)out, ldo, H, V,            \
                                                             gain_per_head, gate_act)
    if (dtype == 0 && wide) SLLM_HNG(float, true);
    else if (dtype == 0) SLLM_HNG(float, false);
    else if (dtype == 1 && wide) SLLM_HNG(bf16, true);
    else if (dtype == 1) SLLM_HNG(bf16, false);
    else return (int)cudaErrorInvalidValue;
#undef SLLM_HNG
    SLLM_LAUNCH_CHECK();
    return 0;
}

SLLM_EXPORT int sllm_lowrank_decay(const float* pre, int64_t ldp, const float* w2t,
                                   const float* w0, const float* a_bias, float decay_scale,
                                   float* out, int n_tokens, int C, int R, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (C <= 0 || R <= 0 || R > 1024 || ldp < C + R) return (int)cudaErrorInvalidValue;
    dim3 grid((C + 255) / 256, (n_tokens + LOWRANK_TOKENS - 1) / LOWRANK_TOKENS);
    if (grid.y > 65535) return (int)cudaErrorInvalidValue;
    lowrank_decay_kernel<<<grid, 256, LOWRANK_TOKENS * R * sizeof(float), stream>>>(
        pre, ldp, w2t, w0, a_bias, decay_scale, out, n_tokens, C, R);
    SLLM_LAUNCH_CHECK();
    return 0;
}

// Up to two products of one `pre` in a launch (n_jobs 1 or 2); per job: col0, w2t [R, C], bias
// (may be null), rate_log with per_rate (mode 1), rate (mode 2), tanh_in, mode, out [N, C], out_dtype (0 = float32,
// 1 = bfloat16), C, R.
SLLM_EXPORT int sllm_lowrank_expand(const float* pre, int64_t ldp, int n_jobs, const int* col0,
                                    const float* const* w2t, const float* const* bias,
                                    const float* const* rate_log, const int* per_rate,
                                    const float* rates, const int* tanh_in, const int* mode,
                                   void* const* out, const int* out_dtype,
                                    const int* C, const int* R, int n_tokens,
                                    cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (n_jobs < 1 || n_jobs > 2) return (int)cudaErrorInvalidValue;
    ExpandJob j[2] = {};
    int max_r = 0, max_c = 0;
    for (int i = 0; i < n_jobs; ++i) {
        if (C[i] <= 0 || R[i] <= 0 || R[i] > 1024 || col0[i] < 0 || ldp < col0[i] + R[i] ||
            mode[i] < 0 || mode[i] > 3 || out_dtype[i] < 0 || out_dtype[i] > 1 ||
            (mode[i] == 1 && (!rate_log[i] || per_rate[i] <= 0 || C[i] % per_rate[i])))
            return (int)cudaErrorInvalidValue;
        j[i].col0 = col0[i]; j[i].w2t = w2t[i]; j[i].bias = bias[i]; j[i].rate_log = rate_log[i];
        j[i].per_rate = per_rate[i]; j[i].mode = mode[i]; j[i].out = out[i];
        j[i].rate = rates[i]; j[i].tanh_in = tanh_in[i];
        j[i].out_bf16 = out_dtype[i]; j[i].C = C[i]; j[i].R = R[i];
        max_r = R[i] > max_r ? R[i] : max_r;
        max_c = C[i] > max_c ? C[i] : max_c;
    }
    // steps of few tokens: narrow CTAs, so that the channels spread over more SMs; long steps: more
    // tokens a CTA and two channels a thread, so that the weights are read less often
    bool wide = n_tokens >= 512;
    for (int i = 0; i < n_jobs; ++i)
        wide = wide && C[i] % 2 == 0 && !(((uintptr_t)w2t[i] | (uintptr_t)out[i]) & 7);
    const int tokens = wide ? 2 * LOWRANK_TOKENS : LOWRANK_TOKENS;
    const int threads = wide ? 128 : n_tokens <= 2 * LOWRANK_TOKENS && max_c >= 1024 ? 64 : 256;
    const int channels = wide ? 2 * threads : threads;
    const int blocks0 = (j[0].C + channels - 1) / channels;
    const int blocks1 = n_jobs > 1 ? (j[1].C + channels - 1) / channels : 0;
    dim3 grid(blocks0 + blocks1, (n_tokens + tokens - 1) / tokens);
    const size_t smem = (size_t)tokens * ((max_r + 3) / 4 * 4) * sizeof(float);
    if (grid.y > 65535) return (int)cudaErrorInvalidValue;
    auto kernel = wide ? lowrank_expand_kernel<2 * LOWRANK_TOKENS, 2, 8>
                       : lowrank_expand_kernel<LOWRANK_TOKENS, 1, 16>;
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                             (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    return (int)sllm_launch_pdl(kernel, grid, dim3(threads), smem, stream, pre, ldp, j[0], j[1],
                                blocks0, n_tokens);
}

// out = parts of o * act(gate) over their root mean squares, times gain; after: parts of o over
// their root mean squares, times gain, times act(gate).  gate_act 0 = silu, 1 = sigmoid.  o: float
// [n_tokens, W]; gate / out: rows ldg / ldo apart.
SLLM_EXPORT int sllm_gate_part_norm(const float* o, const void* gate, int64_t ldg,
                                    const float* gain, float eps, void* out, int64_t ldo,
                                    int n_tokens, int W, int parts, int gate_act, int after,
                                    int dtype, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (W <= 0 || parts < 1 || parts > 65535 || W % parts || ldg < W || ldo < W ||
        gate_act < 0 || gate_act > 1)
        return (int)cudaErrorInvalidValue;
    const int P = W / parts;
    const size_t smem = (size_t)P * sizeof(float);
    if (smem > 160 * 1024) return (int)cudaErrorInvalidValue;
    const bool vec = P % 4 == 0 && ldg % 4 == 0 && ldo % 4 == 0 &&
                     !(((uintptr_t)o | (uintptr_t)gate | (uintptr_t)out) & 15);
    typedef __nv_bfloat16 bf16;
#define SLLM_GPN(T, V)                                                                           \
    do {                                                                                         \
        if (smem > 48 * 1024) {                                                                  \
            cudaError_t e = cudaFuncSetAttribute(gate_part_norm_kernel<T, V>,                    \
                                                 cudaFuncAttributeMaxDynamicSharedMemorySize,    \
                                                 (int)smem);                                     \
            if (e != cudaSuccess) return (int)e;                                                 \
        }                                                                                        \
        return (int)sllm_launch_pdl(gate_part_norm_kernel<T, V>, dim3(n_tokens, parts),          \
                                    dim3(256), smem, stream, o, (const T*)gate, ldg, gain, eps,  \
                                    (T*)out, ldo, W, P, gate_act, after);                                         \
    } while (0)
    if (dtype == 0 && vec) SLLM_GPN(float, 4);
    if (dtype == 0) SLLM_GPN(float, 1);
    if (dtype == 1 && vec) SLLM_GPN(bf16, 4);
    if (dtype == 1) SLLM_GPN(bf16, 1);
#undef SLLM_GPN
    return (int)cudaErrorInvalidValue;
}

SLLM_EXPORT int sllm_ssd_gates(const float* pre, int64_t ldp, const float* bias,
                               const float* A_log, float* log_a, float* b, int n_tokens, int H,
                               cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (H <= 0 || ldp < H) return (int)cudaErrorInvalidValue;
    int64_t blocks = ((int64_t)n_tokens * H + 255) / 256;
    if (blocks > 148 * 16) blocks = 148 * 16;
    return (int)sllm_launch_pdl(ssd_gates_kernel, dim3((int)blocks), dim3(256), 0, stream, pre, ldp,
                                bias, A_log, log_a, b, n_tokens, H);
}

// running: float [slots, H], read and written at the rows' slots.  one_each: no row brings more
// than one token.
SLLM_EXPORT int sllm_memory_gates(const float* pre, int64_t ldp, const float* bi, const float* bf,
                                  float cap, float* running, const int* row_start,
                                  const int* row_slot, float* log_a, float* b, float* floor,
                                  int n_rows, int H, int one_each, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (H <= 0 || ldp < 2 * (int64_t)H || !(cap > 0.f) || n_rows > 65535)
        return (int)cudaErrorInvalidValue;
    MemoryGates a = {pre, ldp, bi, bf, cap, running, row_start, row_slot, log_a, b, floor, H};
    if (one_each)
        return (int)sllm_launch_pdl(memory_gates_step_kernel, dim3((n_rows * H + 127) / 128),
                                    dim3(128), 0, stream, a, n_rows);
    return (int)sllm_launch_pdl(memory_gates_kernel, dim3(H, n_rows), dim3(256), 0, stream, a);
}

// h: [n_tokens, >= d] (dtype), mu: float [M, d], state: float [slots, d], out: [M, n_tokens, d] (dtype).
SLLM_EXPORT int sllm_shift_mix(const void* h, int64_t ldh, const float* mu, int M, float* state,
                               const int* token_row, const int* row_start, const int* row_slot,
                               void* out, int n_tokens, int d, int dtype, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    const int runs = (n_tokens + SHIFT_RUN - 1) / SHIFT_RUN;
    if (d <= 0 || M < 1 || ldh < d || runs > 65535) return (int)cudaErrorInvalidValue;
    const bool vec = ((d | ldh) & 3) == 0 &&
                     !(((uintptr_t)h | (uintptr_t)mu | (uintptr_t)state | (uintptr_t)out) & 15);
    const int per = vec ? 4 : 1;
    const dim3 grid((d / per + 127) / 128, runs);
    typedef __nv_bfloat16 bf16;
#define SLLM_SM(T, V)                                                                              \
    return (int)sllm_launch_pdl(shift_mix_kernel<T, V>, grid, dim3(128), 0, stream, (const T*)h,   \
                                ldh, mu, M, state, token_row, row_start, row_slot, (T*)out, d,     \
                                n_tokens)
    if (dtype == 0 && vec) SLLM_SM(float, 4);
    if (dtype == 0) SLLM_SM(float, 1);
    if (dtype == 1 && vec) SLLM_SM(bf16, 4);
    if (dtype == 1) SLLM_SM(bf16, 1);
#undef SLLM_SM
    return (int)cudaErrorInvalidValue;
}

SLLM_EXPORT int sllm_silu_columns(void* x, int64_t ldx, int n_tokens, int C, int dtype,
                                  cudaStream_t stream) {
    if (n_tokens <= 0 || C == 0) return 0;
    if (C < 0 || ldx < C) return (int)cudaErrorInvalidValue;
    const bool vec = ((C | ldx) & 3) == 0 && !((uintptr_t)x & 15);
    const int64_t items = (int64_t)n_tokens * (vec ? C / 4 : C);
    int64_t blocks = (items + 255) / 256;
    if (blocks > 148 * 32) blocks = 148 * 32;
    typedef __nv_bfloat16 bf16;
#define SLLM_SC(T, V)                                                                              \
    return (int)sllm_launch_pdl(silu_columns_kernel<T, V>, dim3((int)blocks), dim3(256), 0, stream, \
                                (T*)x, ldx, C, items)
    if (dtype == 0 && vec) SLLM_SC(float, 4);
    if (dtype == 0) SLLM_SC(float, 1);
    if (dtype == 1 && vec) SLLM_SC(bf16, 4);
    if (dtype == 1) SLLM_SC(bf16, 1);
#undef SLLM_SC
    return (int)cudaErrorInvalidValue;
}
