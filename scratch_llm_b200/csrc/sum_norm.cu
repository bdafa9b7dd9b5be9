// RMS norms fused with the sum of everything a layer left pending for the residual stream.
//
//   x[n]    = resid[n] + sum_i coef_i * term_i[n]  +  routed(n)          (32-bit)
//   outA[n] = x[n] / sqrt(mean(x[n]^2) + eps) * gA,   outB[n] likewise with gB (optional)
//
// Two outputs serve layers whose branches run side by side behind a norm each: both norms have
// the same x, so one pass over the stream gives both.  routed(n) (optional) is what a routed
// feed-forward has not added up yet: sum over the token's choices, in their order, of weight *
// (the expert's output row), plus sigmoid(gate) * (the shared expert's output).
// Without out_rows every token is normed and the stream is updated in place; with out_rows only
// the listed tokens are normed (outA is then [rows, d]) and the stream is not written.
// One CTA per token; the row waits in shared memory between the two passes, so a token's result
// does not depend on its neighbours.
#include "few.cuh"

namespace sllm {

constexpr int SN_MAX_TERMS = 4;

struct SumNorm {
    float* resid;
    const void* term[SN_MAX_TERMS]; float coef[SN_MAX_TERMS]; int n_terms;
    RoutedRows routed;
    const float* gA; const float* gB; float eps;
    void* outA; void* outB;
    const int* out_rows; int d;
};

template <typename T, int V>
__global__ void __launch_bounds__(512) sum_norm_kernel(const SumNorm a) {
    extern __shared__ __align__(16) float row[];      // [d]
    __shared__ float scratch[33];
    pdl_wait();
    pdl_trigger();
    const int d = a.d;
    const int64_t n = a.out_rows ? a.out_rows[blockIdx.x] : blockIdx.x;
    float* r = a.resid + n * d;
    const bool keep = a.out_rows == nullptr && (a.n_terms > 0 || a.routed.y != nullptr);
    const float fs = shared_factor(a.routed, n);
    float ss = 0.f;
    for (int c = threadIdx.x * V; c < d; c += blockDim.x * V) {
        Few<V> x = few<V>(r + c);
#pragma unroll
        for (int i = 0; i < SN_MAX_TERMS; ++i)
            if (i < a.n_terms) {
                const Few<V> t = few<V>(reinterpret_cast<const T*>(a.term[i]) + n * d + c);
#pragma unroll
                for (int k = 0; k < V; ++k) x.v[k] = fmaf(a.coef[i], t.v[k], x.v[k]);
            }
        if (a.routed.y) {
            const Few<V> sum = routed_sum<T, V>(a.routed, n, d, c, fs);
#pragma unroll
            for (int k = 0; k < V; ++k) x.v[k] += sum.v[k];
        }
        if (keep) put<V>(r + c, x);
        put<V>(row + c, x);
#pragma unroll
        for (int k = 0; k < V; ++k) ss = fmaf(x.v[k], x.v[k], ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)d + a.eps);
    T* oA = reinterpret_cast<T*>(a.outA) + (int64_t)blockIdx.x * d;
    T* oB = a.outB ? reinterpret_cast<T*>(a.outB) + (int64_t)blockIdx.x * d : nullptr;
    for (int c = threadIdx.x * V; c < d; c += blockDim.x * V) {
        const Few<V> x = few<V>(row + c), g = few<V>(a.gA + c);
        Few<V> y;
#pragma unroll
        for (int k = 0; k < V; ++k) y.v[k] = x.v[k] * inv * g.v[k];
        put<V>(oA + c, y);
        if (oB) {
            const Few<V> h = few<V>(a.gB + c);
#pragma unroll
            for (int k = 0; k < V; ++k) y.v[k] = x.v[k] * inv * h.v[k];
            put<V>(oB + c, y);
        }
    }
}

// out[n, :] = table[id] * scale + pairs[row], the stream's start for designs whose embedding adds
// a vector for the pair (previous token, token): row = (previous * mul_prev + id * mul_cur) mod
// buckets, and row `buckets` for a sequence's first token.  The previous token of a row's first
// token is in last[slot], where the row's last token is left for the next step (by the block of
// the row's first token, after it has read the old one).  ids as in embed_kernel (-1 - j stands
// for pending[j]).  Padding tokens (token_row -1) take row `buckets`.  One block per token.
// V: elements per access (4 where d allows it, else 1).
template <typename T, int V>
__global__ void embed_pair_kernel(const int* __restrict__ ids, const int* __restrict__ pending,
                                  const int* __restrict__ positions,
                                  const int* __restrict__ token_row,
                                  const int* __restrict__ row_start,
                                  const int* __restrict__ row_slot, const T* __restrict__ table,
                                  const T* __restrict__ pairs, int* __restrict__ last,
                                  int64_t mul_prev, int64_t mul_cur, int64_t buckets, float scale,
                                  float* __restrict__ out, int d) {
    pdl_wait();
    pdl_trigger();
    const int n = blockIdx.x;
    int id = ids[n];
    if (id < 0) id = pending[-1 - id];
    const int r = token_row[n];
    int64_t pair = buckets;
    if (r >= 0) {
        const int t0 = row_start[r];
        int prev;
        if (n > t0) {
            prev = ids[n - 1];
            if (prev < 0) prev = pending[-1 - prev];
        } else {
            int* mine = last + row_slot[r];
            prev = *mine;
            __syncthreads();               // every thread has read it
            if (threadIdx.x == 0) {
                int end = ids[row_start[r + 1] - 1];
                if (end < 0) end = pending[-1 - end];
                *mine = end;
            }
        }
        if (positions[n] > 0) pair = ((int64_t)prev * mul_prev + (int64_t)id * mul_cur) % buckets;
    }
    const T* a = table + (int64_t)id * d;
    const T* b = pairs + pair * d;
    float* dst = out + (int64_t)n * d;
    for (int i = threadIdx.x * V; i < d; i += blockDim.x * V) {
        const Few<V> x = few<V>(a + i), y = few<V>(b + i);
        Few<V> z;
#pragma unroll
        for (int k = 0; k < V; ++k) z.v[k] = fmaf(x.v[k], scale, y.v[k]);
        put<V>(dst + i, z);
    }
}

}  // namespace sllm

using namespace sllm;

// dtype (of the terms, of shared and of the outputs): 0 = float32, 1 = bfloat16.  out_rows (may
// be null): int [n_out].  gB / outB may be null.
SLLM_EXPORT int sllm_sum_norm(float* resid, const void* const* terms, const float* coefs,
                              int n_terms, const float* y, const int* ids, const float* weights,
                              const int* place, int top, const void* shared, const float* sg,
                              int64_t ldsg, const float* gA, const float* gB, float eps, void* outA,
                              void* outB, const int* out_rows, int n_out, int d, int dtype,
                              cudaStream_t stream) {
    if (n_out <= 0) return 0;
    if (d <= 0 || d > 32768 || n_terms < 0 || n_terms > SN_MAX_TERMS || (y && top < 1) ||
        (gB == nullptr) != (outB == nullptr))
        return (int)cudaErrorInvalidValue;
    SumNorm a = {};
    a.resid = resid;
    a.n_terms = n_terms;
    uintptr_t bits = (uintptr_t)resid | (uintptr_t)gA | (uintptr_t)gB | (uintptr_t)outA |
                     (uintptr_t)outB | (uintptr_t)y | (uintptr_t)shared;
    for (int i = 0; i < n_terms; ++i) {
        a.term[i] = terms[i];
        a.coef[i] = coefs[i];
        bits |= (uintptr_t)terms[i];
    }
    a.routed = RoutedRows{y, ids, weights, place, top, shared, sg, ldsg};
    a.gA = gA; a.gB = gB; a.eps = eps; a.outA = outA; a.outB = outB;
    a.out_rows = out_rows; a.d = d;
    const bool vec = d % 4 == 0 && !(bits & 15);
    const size_t smem = (size_t)d * sizeof(float);
    int threads = 64;
    while (threads < 512 && threads * (vec ? 4 : 1) < d) threads <<= 1;
#define SLLM_SN(T, V)                                                                             \
    do {                                                                                          \
        if (smem > 48 * 1024) {                                                                   \
            cudaError_t e = cudaFuncSetAttribute(sum_norm_kernel<T, V>,                           \
                                                 cudaFuncAttributeMaxDynamicSharedMemorySize,     \
                                                 (int)smem);                                      \
            if (e != cudaSuccess) return (int)e;                                                  \
        }                                                                                         \
        return (int)sllm_launch_pdl(sum_norm_kernel<T, V>, dim3(n_out), dim3(threads), smem,      \
                                    stream, a);                                                   \
    } while (0)
    if (dtype == 0 && vec) SLLM_SN(float, 4);
    if (dtype == 0) SLLM_SN(float, 1);
    if (dtype == 1 && vec) SLLM_SN(__nv_bfloat16, 4);
    if (dtype == 1) SLLM_SN(__nv_bfloat16, 1);
#undef SLLM_SN
    return (int)cudaErrorInvalidValue;
}

// table [vocab, d], pairs [buckets + 1, d] (dtype), last: int [slots].
SLLM_EXPORT int sllm_embed_pair(const int* ids, const int* pending, const int* positions,
                                const int* token_row, const int* row_start, const int* row_slot,
                                const void* table, const void* pairs, int* last, int64_t mul_prev,
                                int64_t mul_cur, int64_t buckets, float scale, float* out,
                                int n_tokens, int d, int dtype, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (d <= 0 || buckets < 1 || mul_prev < 0 || mul_cur < 0) return (int)cudaErrorInvalidValue;
    const int threads = d >= 1024 ? 256 : 64;
    const bool vec = d % 4 == 0 && !(((uintptr_t)table | (uintptr_t)pairs | (uintptr_t)out) & 15);
#define SLLM_EP(T, V)                                                                              \
    return (int)sllm_launch_pdl(embed_pair_kernel<T, V>, dim3(n_tokens), dim3(threads), 0, stream, \
                                ids, pending, positions, token_row, row_start, row_slot,          \
                                (const T*)table, (const T*)pairs, last, mul_prev, mul_cur,        \
                                buckets, scale, out, d)
    if (dtype == 0 && vec) SLLM_EP(float, 4);
    if (dtype == 0) SLLM_EP(float, 1);
    if (dtype == 1 && vec) SLLM_EP(__nv_bfloat16, 4);
    if (dtype == 1) SLLM_EP(__nv_bfloat16, 1);
#undef SLLM_EP
    return (int)cudaErrorInvalidValue;
}
