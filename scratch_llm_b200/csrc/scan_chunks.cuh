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

// ---- tensor-core pieces of the chunk kernels (bfloat16)

typedef __nv_bfloat16 bf16;
constexpr int PARTS = 3;        // bfloat16 parts of a 32-bit operand: they hold all of its 24 bits

__device__ __forceinline__ uint32_t smem_addr(const void* p) {
    return (uint32_t)__cvta_generic_to_shared(p);
}
__device__ __forceinline__ void ldsm4(uint32_t* r, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm2(uint32_t* r, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];"
                 : "=r"(r[0]), "=r"(r[1]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4_t(uint32_t* r, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm2_t(uint32_t* r, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];"
                 : "=r"(r[0]), "=r"(r[1]) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float* c, const uint32_t* a, const uint32_t* b) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, "
                 "{%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}
// The PARTS parts of two 32-bit numbers, each part a pair of bfloat16.
__device__ __forceinline__ void split2(float x, float y, uint32_t* part) {
#pragma unroll
    for (int p = 0; p < PARTS; ++p) {
        const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
        part[p] = *reinterpret_cast<const uint32_t*>(&h);
        x -= __low2float(h);
        y -= __high2float(h);
    }
}

}  // namespace sllm
