// V values at a time (4: 16- or 8-byte accesses, suitably aligned; 1: one by one), widened to
// 32-bit, and what a routed feed-forward has not added up yet, for the kernels that add it up while
// they read the residual stream.
#pragma once

#include "common.cuh"

namespace sllm {

template <int V> struct Few { float v[V]; };
template <int V> __device__ __forceinline__ Few<V> few(const float* p) {
    Few<V> r;
    if (V == 4) {
        const float4 x = *reinterpret_cast<const float4*>(p);
        r.v[0] = x.x; r.v[V - 3] = x.y; r.v[V - 2] = x.z; r.v[V - 1] = x.w;
    } else {
        r.v[0] = *p;
    }
    return r;
}
template <int V> __device__ __forceinline__ Few<V> few(const __nv_bfloat16* p) {
    Few<V> r;
    if (V == 4) {
        const uint2 x = *reinterpret_cast<const uint2*>(p);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&x);
        r.v[0] = __low2float(h[0]); r.v[V - 3] = __high2float(h[0]);
        r.v[V - 2] = __low2float(h[1]); r.v[V - 1] = __high2float(h[1]);
    } else {
        r.v[0] = __bfloat162float(*p);
    }
    return r;
}
template <int V> __device__ __forceinline__ void put(float* p, const Few<V>& r) {
    if (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[V - 3], r.v[V - 2], r.v[V - 1]);
    else *p = r.v[0];
}
template <int V> __device__ __forceinline__ void put(__nv_bfloat16* p, const Few<V>& r) {
    if (V == 4) {
        uint2 x;
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&x);
        h[0] = __floats2bfloat162_rn(r.v[0], r.v[V - 3]);
        h[1] = __floats2bfloat162_rn(r.v[V - 2], r.v[V - 1]);
        *reinterpret_cast<uint2*>(p) = x;
    } else {
        *p = __float2bfloat16_rn(r.v[0]);
    }
}

// A routed feed-forward's output before it is added up (y null: none): y [places, d], ids / weights /
// place [tokens, top]; shared [tokens, d] (T, may be null), its gate's logit sg (may be null).
struct RoutedRows {
    const float* y; const int* ids; const float* weights; const int* place; int top;
    const void* shared; const float* sg; int64_t ldsg;
};
// The factor of token n's shared output.
__device__ __forceinline__ float shared_factor(const RoutedRows& a, int64_t n) {
    return a.y && a.shared && a.sg ? 1.0f / (1.0f + expf(-a.sg[n * a.ldsg])) : 1.f;
}
// Columns c .. c + V - 1 of token n's sum: its choices in their order, then the shared output.
template <typename T, int V>
__device__ __forceinline__ Few<V> routed_sum(const RoutedRows& a, int64_t n, int d, int c, float fs) {
    Few<V> sum;
#pragma unroll
    for (int k = 0; k < V; ++k) sum.v[k] = 0.f;
    for (int j = 0; j < a.top; ++j) {
        const int p = a.place[n * a.top + j];
        if (p < 0) continue;
        const float w = a.weights[n * a.top + j];
        const Few<V> t = few<V>(a.y + (int64_t)p * d + c);
#pragma unroll
        for (int k = 0; k < V; ++k) sum.v[k] = fmaf(w, t.v[k], sum.v[k]);
    }
    if (a.shared) {
        const Few<V> t = few<V>(reinterpret_cast<const T*>(a.shared) + n * d + c);
#pragma unroll
        for (int k = 0; k < V; ++k) sum.v[k] = fmaf(fs, t.v[k], sum.v[k]);
    }
    return sum;
}

}  // namespace sllm
