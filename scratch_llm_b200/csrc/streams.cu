// A residual stream of several parts (hyper-connections): S parts x_1 .. x_S per token instead of one
// sum, fused with the norm in front of the next sublayer.
//
//   update  x_t <- sum_s mix[s, t] x_s + out[t] y        (every part from all old ones at once)
//           with y what the sublayer before left pending: sum_i coef_i * term_i + routed
//   read    u = sum_s in[s] x_s                           (in null: the plain sum)
//   norm    out = (u - mean) / sqrt(var + eps) * gain + bias, or u / sqrt(mean(u^2) + eps) * gain
//           (rms); bias may be null
//
// One pass: a sublayer's update, the next sublayer's reading and its norm are one launch, and each
// part is read and written once.  The parts are [tokens, S, d], all arithmetic is 32-bit; the terms
// are branch outputs in the compute dtype.  Without out_rows every token is normed and the parts are
// updated in place; with out_rows only the listed tokens are (out is then [rows, d]) and the parts
// are not written.  One CTA per token; u waits in shared memory between the passes, so a token's
// result does not depend on its neighbours.
#include "few.cuh"

namespace sllm {

constexpr int ST_MAX_TERMS = 4;
constexpr int ST_MAX_STREAMS = 16;

struct StreamsNorm {
    float* parts;                                   // [tokens, S, d]
    int S;
    int update;                                     // 0: nothing is pending
    const void* term[ST_MAX_TERMS]; float coef[ST_MAX_TERMS]; int n_terms;
    RoutedRows routed;
    const float* mix; const float* to;              // [S, S] (from, to), [S]
    const float* from;                              // [S] or null
    const float* gain; const float* bias; float eps; int rms;
    void* out;
    const int* out_rows; int d;
};

// S: the number of parts, or 0 for any number up to ST_MAX_STREAMS.  V: elements per access.
template <typename T, int V, int S>
__global__ void __launch_bounds__(512) streams_norm_kernel(const StreamsNorm a) {
    constexpr int MAXS = S ? S : ST_MAX_STREAMS;
    extern __shared__ __align__(16) float row[];    // [d]
    __shared__ float scratch[33];
    __shared__ float mix[MAXS * MAXS], to[MAXS], from[MAXS];
    const int n_parts = S ? S : a.S;
    if (a.update)
        for (int i = threadIdx.x; i < n_parts * n_parts; i += blockDim.x) {
            mix[i] = a.mix[i];
            if (i < n_parts) to[i] = a.to[i];
        }
    if (threadIdx.x < n_parts) from[threadIdx.x] = a.from ? a.from[threadIdx.x] : 1.f;
    __syncthreads();
    pdl_wait();
    pdl_trigger();
    const int d = a.d;
    const int64_t n = a.out_rows ? a.out_rows[blockIdx.x] : blockIdx.x;
    float* base = a.parts + n * n_parts * d;
    const bool keep = a.out_rows == nullptr;
    const float fs = shared_factor(a.routed, n);
    float sum = 0.f;
    for (int c = threadIdx.x * V; c < d; c += blockDim.x * V) {
        Few<V> x[MAXS];
#pragma unroll
        for (int s = 0; s < MAXS; ++s)
            if (s < n_parts) x[s] = few<V>(base + (int64_t)s * d + c);
        Few<V> u;
#pragma unroll
        for (int k = 0; k < V; ++k) u.v[k] = 0.f;
        if (a.update) {
            Few<V> y;
#pragma unroll
            for (int k = 0; k < V; ++k) y.v[k] = 0.f;
            if (a.routed.y) y = routed_sum<T, V>(a.routed, n, d, c, fs);
#pragma unroll
            for (int i = 0; i < ST_MAX_TERMS; ++i)
                if (i < a.n_terms) {
                    const Few<V> t = few<V>(reinterpret_cast<const T*>(a.term[i]) + n * d + c);
#pragma unroll
                    for (int k = 0; k < V; ++k) y.v[k] = fmaf(a.coef[i], t.v[k], y.v[k]);
                }
#pragma unroll (S ? S : 1)
            for (int t = 0; t < MAXS; ++t)
                if (t < n_parts) {
                    Few<V> z;
#pragma unroll
                    for (int k = 0; k < V; ++k) z.v[k] = to[t] * y.v[k];
#pragma unroll
                    for (int s = 0; s < MAXS; ++s)
                        if (s < n_parts) {
                            const float w = mix[s * n_parts + t];
#pragma unroll
                            for (int k = 0; k < V; ++k) z.v[k] = fmaf(w, x[s].v[k], z.v[k]);
                        }
                    if (keep) put<V>(base + (int64_t)t * d + c, z);
#pragma unroll
                    for (int k = 0; k < V; ++k) u.v[k] = fmaf(from[t], z.v[k], u.v[k]);
                }
        } else {
#pragma unroll
            for (int s = 0; s < MAXS; ++s)
                if (s < n_parts)
#pragma unroll
                    for (int k = 0; k < V; ++k) u.v[k] = fmaf(from[s], x[s].v[k], u.v[k]);
        }
        put<V>(row + c, u);
#pragma unroll
        for (int k = 0; k < V; ++k) sum += a.rms ? u.v[k] * u.v[k] : u.v[k];
    }
    sum = block_sum(sum, scratch) / (float)d;
    float mean = 0.f, var = sum;
    if (!a.rms) {
        mean = sum;
        float dev = 0.f;
        for (int c = threadIdx.x * V; c < d; c += blockDim.x * V) {
            const Few<V> x = few<V>(row + c);
#pragma unroll
            for (int k = 0; k < V; ++k) dev = fmaf(x.v[k] - mean, x.v[k] - mean, dev);
        }
        var = block_sum(dev, scratch) / (float)d;
    }
    const float inv = 1.0f / sqrtf(var + a.eps);
    T* o = reinterpret_cast<T*>(a.out) + (int64_t)blockIdx.x * d;
    for (int c = threadIdx.x * V; c < d; c += blockDim.x * V) {
        const Few<V> x = few<V>(row + c), g = few<V>(a.gain + c);
        Few<V> y;
#pragma unroll
        for (int k = 0; k < V; ++k) y.v[k] = (x.v[k] - mean) * inv * g.v[k];
        if (a.bias) {
            const Few<V> b = few<V>(a.bias + c);
#pragma unroll
            for (int k = 0; k < V; ++k) y.v[k] += b.v[k];
        }
        put<V>(o + c, y);
    }
}

}  // namespace sllm

using namespace sllm;

SLLM_EXPORT int sllm_streams_max() { return ST_MAX_STREAMS; }

// parts: float [n_tokens, S, d].  mix [S, S] (from, to) and to [S]: null together when nothing is
// pending.  terms, routed: as sllm_sum_norm.  from [S], bias [d], out_rows [n_out]: may be null.
// dtype (of the terms, of shared and of out): 0 = float32, 1 = bfloat16.
SLLM_EXPORT int sllm_streams_norm(float* parts, int S, const float* mix, const float* to,
                                  const void* const* terms, const float* coefs, int n_terms,
                                  const float* y, const int* ids, const float* weights,
                                  const int* place, int top, const void* shared, const float* sg,
                                  int64_t ldsg, const float* from, const float* gain,
                                  const float* bias, float eps, int rms, void* out,
                                  const int* out_rows, int n_out, int d, int dtype,
                                  cudaStream_t stream) {
    if (n_out <= 0) return 0;
    if (d <= 0 || d > 32768 || S < 1 || S > ST_MAX_STREAMS || n_terms < 0 ||
        n_terms > ST_MAX_TERMS || (y && top < 1) || (mix == nullptr) != (to == nullptr) ||
        (!mix && (n_terms || y)))
        return (int)cudaErrorInvalidValue;
    StreamsNorm a = {};
    a.parts = parts; a.S = S; a.update = mix != nullptr; a.n_terms = n_terms;
    uintptr_t bits = (uintptr_t)parts | (uintptr_t)gain | (uintptr_t)bias | (uintptr_t)out |
                     (uintptr_t)y | (uintptr_t)shared;
    for (int i = 0; i < n_terms; ++i) {
        a.term[i] = terms[i];
        a.coef[i] = coefs[i];
        bits |= (uintptr_t)terms[i];
    }
    a.routed = RoutedRows{y, ids, weights, place, top, shared, sg, ldsg};
    a.mix = mix; a.to = to; a.from = from; a.gain = gain; a.bias = bias; a.eps = eps; a.rms = rms;
    a.out = out; a.out_rows = out_rows; a.d = d;
    const bool vec = d % 4 == 0 && !(bits & 15);
    const size_t smem = (size_t)d * sizeof(float);
    int threads = 64;
    while (threads < 512 && threads * (vec ? 4 : 1) < d) threads <<= 1;
#define SLLM_ST(T, V, NS)                                                                         \
    do {                                                                                          \
        if (smem > 44 * 1024) {                                                                   \
            cudaError_t e = cudaFuncSetAttribute(streams_norm_kernel<T, V, NS>,                   \
                                                 cudaFuncAttributeMaxDynamicSharedMemorySize,     \
                                                 (int)smem);                                      \
            if (e != cudaSuccess) return (int)e;                                                  \
        }                                                                                         \
        return (int)sllm_launch_pdl(streams_norm_kernel<T, V, NS>, dim3(n_out), dim3(threads),    \
                                    smem, stream, a);                                             \
    } while (0)
#define SLLM_ST_V(T, V)                                                                           \
    do {                                                                                          \
        if (S == 1) SLLM_ST(T, V, 1);                                                             \
        if (S == 2) SLLM_ST(T, V, 2);                                                             \
        if (S == 3) SLLM_ST(T, V, 3);                                                             \
        if (S == 4) SLLM_ST(T, V, 4);                                                             \
        SLLM_ST(T, 1, 0);                                                                         \
    } while (0)
    if (dtype == 0 && vec) SLLM_ST_V(float, 4);
    if (dtype == 0) SLLM_ST_V(float, 1);
    if (dtype == 1 && vec) SLLM_ST_V(__nv_bfloat16, 4);
    if (dtype == 1) SLLM_ST_V(__nv_bfloat16, 1);
#undef SLLM_ST_V
#undef SLLM_ST
    return (int)cudaErrorInvalidValue;
}
