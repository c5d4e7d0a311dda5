// bf16_split.cuh — an F32 number as the sum of two BF16 values (about 16 mantissa bits), the operand form of the tensor-core GEMM
// (prefill_gemm.cu): workspace [hi: Mp x K][lo: Mp x K], Mp = rows rounded up to 128.
#pragma once
#include <cuda_bf16.h>
#include <cstdint>
#include <cstddef>

namespace nt { namespace b200 {

__device__ __forceinline__ void split_store1(__nv_bfloat16* hi, __nv_bfloat16* lo, size_t i, float v) {
    const __nv_bfloat16 h = __float2bfloat16_rn(v);
    hi[i] = h;
    lo[i] = __float2bfloat16_rn(v - __bfloat162float(h));
}
// four consecutive numbers, i a multiple of 4
__device__ __forceinline__ void split_store4(__nv_bfloat16* hi, __nv_bfloat16* lo, size_t i, const float (&v)[4]) {
    __nv_bfloat162 h[2], l[2];
#pragma unroll
    for (int e = 0; e < 2; e++) {
        h[e] = __floats2bfloat162_rn(v[2 * e], v[2 * e + 1]);
        const float2 f = __bfloat1622float2(h[e]);
        l[e] = __floats2bfloat162_rn(v[2 * e] - f.x, v[2 * e + 1] - f.y);
    }
    *reinterpret_cast<uint2*>(hi + i) = make_uint2(*reinterpret_cast<const uint32_t*>(&h[0]), *reinterpret_cast<const uint32_t*>(&h[1]));
    *reinterpret_cast<uint2*>(lo + i) = make_uint2(*reinterpret_cast<const uint32_t*>(&l[0]), *reinterpret_cast<const uint32_t*>(&l[1]));
}
// where the lo half of a split workspace of M rows x K columns starts, in 16-bit words
__host__ __device__ __forceinline__ size_t split_lo_offset(int M, int K) { return ((size_t)M + 127) / 128 * 128 * (size_t)K; }

}}  // namespace nt::b200
