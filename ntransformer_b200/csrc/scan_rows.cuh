// scan_rows.cuh — pieces shared by the recurrences over the rows of a step (wkv.cu, mlstm.cu): asynchronous staging copies and the joint reduction
// of a tile's dot products.
#pragma once
#include <cuda_runtime.h>
#include <cstdint>

namespace nt { namespace b200 {

constexpr int SCAN_TILE = 16;      // rows per staged tile

__device__ __forceinline__ void cp_async16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

// part[0..15] (one number per row and lane) -> sums over the LN lanes of a column: afterwards lane l holds, in part[0..N-1], the rows
// first_row .. first_row + N - 1.  Every step halves the rows a lane is responsible for and sends the other half to its partner.
template <int LN>
__device__ __forceinline__ int reduce_rows(float (&part)[SCAN_TILE], int l) {
    int base = 0;
    constexpr int STEPS = LN == 1 ? 0 : LN == 2 ? 1 : LN == 4 ? 2 : LN == 8 ? 3 : LN == 16 ? 4 : 5;
#pragma unroll
    for (int s = 0; s < STEPS; s++) {
        const int m = LN >> (s + 1);
        const bool hi = (l & m) != 0;
        if (s < 4) {
            const int half = SCAN_TILE >> (s + 1);
#pragma unroll
            for (int j = 0; j < SCAN_TILE / 2; j++) {
                if (j < half) {
                    const float send = hi ? part[j] : part[j + half], keep = hi ? part[j + half] : part[j];
                    part[j] = keep + __shfl_xor_sync(0xFFFFFFFFu, send, m);
                }
            }
            base += hi ? half : 0;
        } else part[0] += __shfl_xor_sync(0xFFFFFFFFu, part[0], m);
    }
    return base;
}

}}  // namespace nt::b200
