// How the chunk kernels of the scans find their chunk: chunks of TC tokens, counted from each row's
// first token of the step.  The chunk that starts at token t of the batch, in row r, has slot
// t / TC + r (distinct for distinct chunks, whatever the rows' lengths), so a launch over slots finds
// its chunk on the device and nothing is read on the host.  n tokens in R rows have slots below
// n / TC + R + 1.
#pragma once

#include "common.cuh"

namespace sllm {

constexpr int TC = 64;          // tokens of a chunk

// The row, its first token and count, and the chunk's first token within the row, of chunk slot `s`;
// false: no chunk has it.  Rows of fewer than `min_chunked` tokens have no chunks.
__device__ __forceinline__ bool find_chunk(const int* row_start, int n_rows, int min_chunked, int s,
                                           int& row, int& t0, int& c0, int& n_new) {
    const int lane = threadIdx.x & 31;
    for (int r0 = 0; r0 < n_rows; r0 += 32) {
        const int r = r0 + lane;
        bool mine = false;
        int start = 0, count = 0;
        if (r < n_rows) {
            start = row_start[r];
            count = row_start[r + 1] - start;
            const int first = start / TC + r;
            mine = count >= min_chunked && s >= first && (s - first) * TC < count;
        }
        const unsigned hit = __ballot_sync(0xffffffffu, mine);
        if (hit) {
            const int who = __ffs(hit) - 1;
            row = r0 + who;
            t0 = __shfl_sync(0xffffffffu, start, who);
            n_new = __shfl_sync(0xffffffffu, count, who);
            c0 = (s - (t0 / TC + row)) * TC;
            return true;
        }
    }
    return false;
}

__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
    return make_float4(__low2float(h[0]), __high2float(h[0]), __low2float(h[1]), __high2float(h[1]));
}

}  // namespace sllm
