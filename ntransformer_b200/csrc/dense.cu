// dense.cu — GEMV / GEMM over dense weight rows (F32, F16, BF16) with F32 activations and F32 accumulation, plus the
// elementwise pieces of the layer-spec model families (engine/layer_spec.h).
//
//   gemv_dense   decode: up to 3 matrices share one activation vector staged once per CTA in shared memory; a warp streams one
//                output row with 16-byte loads; the prologue can RMS-normalise the staged vector; epilogues fuse the residual (+ per-channel gain) and the gated activations, so a
//                decode step needs no separate add / scale / activation launch.
//   gemv_multi   decode: several matrices with an input vector each (and an activation on their rows) in one launch
//   gemv_sum     decode: y (+)= the sum of several matrix-vector products with inputs of their own, routed experts among them: the last
//                products of a block whose mixer and feed-forward join the residual together
//   gemm_dense   prompt tokens on CUDA cores: 64x64x16 tiles, 4x4 outputs per thread, true FP32 FMA.  It serves the exact
//                32-bit mode and shapes the tcgen05 tiles of prefill_gemm.cu do not cover (rows % 128, cols % 64).
// This file is compiled WITHOUT --use_fast_math (tanh / exp / division at full precision): the 32-bit mode depends on it.
#include "kernels_internal.h"
#include "bf16_split.cuh"
#include "ring.cuh"
#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <algorithm>

namespace nt { namespace b200 {

namespace {

__device__ __forceinline__ float gelu_tanh_f(float z) {
    return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }
// z > 0: a z^2 + z / 2;  z <= 0: (1/2 + b)(e^z - 1 - z) + z / 2   (a, b: softplus of the layer's two numbers)
__device__ __forceinline__ float xielu_f(float z, float a, float b) { return z > 0.f ? fmaf(a * z, z, 0.5f * z) : fmaf(0.5f + b, expm1f(z) - z, 0.5f * z); }

template <typename T> struct Elem;
template <> struct Elem<float> {
    static constexpr int PER16 = 4;
    static __device__ __forceinline__ float one(const void* row, int i) { return __ldg(static_cast<const float*>(row) + i); }
    static __device__ __forceinline__ void unpack(const uint4& w, float* f) { f[0] = __uint_as_float(w.x); f[1] = __uint_as_float(w.y); f[2] = __uint_as_float(w.z); f[3] = __uint_as_float(w.w); }
};
template <> struct Elem<__half> {
    static constexpr int PER16 = 8;
    static __device__ __forceinline__ float one(const void* row, int i) { return __half2float(__ushort_as_half(__ldg(static_cast<const unsigned short*>(row) + i))); }
    static __device__ __forceinline__ void unpack(const uint4& w, float* f) {
        const unsigned u[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
        for (int k = 0; k < 4; k++) { float2 p = __half22float2(*reinterpret_cast<const __half2*>(&u[k])); f[2 * k] = p.x; f[2 * k + 1] = p.y; }
    }
};
template <> struct Elem<__nv_bfloat16> {
    static constexpr int PER16 = 8;
    static __device__ __forceinline__ float one(const void* row, int i) { return __uint_as_float((unsigned)__ldg(static_cast<const unsigned short*>(row) + i) << 16); }
    static __device__ __forceinline__ void unpack(const uint4& w, float* f) {
        const unsigned u[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
        for (int k = 0; k < 4; k++) { f[2 * k] = __uint_as_float(u[k] << 16); f[2 * k + 1] = __uint_as_float(u[k] & 0xFFFF0000u); }
    }
};

__device__ __forceinline__ uint4 ld_stream16(const void* p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}

// element r of every stream of one token: X[t][r] <- sum_s M[s][t] X[s][r] + b[t] * v  (all t from the old values)
__device__ __forceinline__ void streams_update(const StreamsIO& sio, int N, int r, float v) {
    float xv[16], nv[16];
#pragma unroll
    for (int s = 0; s < 16; s++) xv[s] = s < sio.S ? sio.X_out[(size_t)s * N + r] : 0.f;
#pragma unroll
    for (int t = 0; t < 16; t++) {
        float acc = 0.f;
        if (t < sio.S) {
#pragma unroll
            for (int s = 0; s < 16; s++) if (s < sio.S) acc = fmaf(sio.M[s * sio.S + t], xv[s], acc);
            acc = fmaf(sio.b[t], v, acc);
        }
        nv[t] = acc;
    }
#pragma unroll
    for (int t = 0; t < 16; t++) if (t < sio.S) sio.X_out[(size_t)t * N + r] = nv[t];
}

struct DenseMats {
    const unsigned char* W[DENSE_MAX_MATS];
    float* y[DENSE_MAX_MATS];
    int out[DENSE_MAX_MATS];
    size_t pitch[DENSE_MAX_MATS];
    int n;
};

constexpr int DV_WARPS = 8;

// <row, xs> for one row, this lane's share; vec: row base and pitch 16-byte aligned and K a multiple of PER16
template <typename T>
__device__ __forceinline__ float dense_row_part(const unsigned char* row, const float* xs, int K, int lane, bool vec) {
    float acc = 0.f;
    constexpr int P = Elem<T>::PER16;
    if (vec) {
        const int nv = K / P;
        int v = lane;
        for (; v + 96 < nv; v += 128) {
            uint4 w[4];
#pragma unroll
            for (int u = 0; u < 4; u++) w[u] = ld_stream16(row + (size_t)(v + 32 * u) * 16);
#pragma unroll
            for (int u = 0; u < 4; u++) {
                float f[P];
                Elem<T>::unpack(w[u], f);
                const float* xp = xs + (size_t)(v + 32 * u) * P;
#pragma unroll
                for (int k = 0; k < P; k++) acc = fmaf(f[k], xp[k], acc);
            }
        }
        for (; v < nv; v += 32) {
            float f[P];
            Elem<T>::unpack(ld_stream16(row + (size_t)v * 16), f);
            const float* xp = xs + (size_t)v * P;
#pragma unroll
            for (int k = 0; k < P; k++) acc = fmaf(f[k], xp[k], acc);
        }
    } else {
        for (int i = lane; i < K; i += 32) acc = fmaf(Elem<T>::one(row, i), xs[i], acc);
    }
    return acc;
}
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, o);
    return v;
}
template <typename T>
__device__ __forceinline__ float dense_row_dot(const unsigned char* row, const float* xs, int K, int lane, bool vec) {
    return warp_sum(dense_row_part<T>(row, xs, K, lane, vec));
}

template <typename T>
__global__ void __launch_bounds__(DV_WARPS * 32) gemv_dense_kernel(DenseMats m, const float* __restrict__ x, int K, int ep,
                                                                   const float* __restrict__ row_scale, float alpha, int vec,
                                                                   const float* __restrict__ norm_w, float eps, StreamsIO sio, int norm_groups) {
    extern __shared__ __align__(16) float xs[];
    __shared__ float red[DV_WARPS];
    __shared__ float inv_g[DENSE_MAX_NORM_GROUPS];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    pdl_launch_dependents();
    pdl_wait();
    float ss = 0.f;
    for (int i = threadIdx.x; i < K; i += DV_WARPS * 32) {
        float v;
        if (sio.X_in) {                   // the blend of the token's residual streams
            v = 0.f;
            for (int st = 0; st < sio.S; st++) { const float xv = sio.X_in[(size_t)st * K + i]; v = sio.a ? fmaf(sio.a[st], xv, v) : v + xv; }
        } else v = x[i];
        xs[i] = v; ss = fmaf(v, v, ss);
    }
    if (norm_w && norm_groups > 1) {        // every run of K / norm_groups channels has its own root mean square: a warp per run
        __syncthreads();
        const int per = K / norm_groups;
        for (int g = warp; g < norm_groups; g += DV_WARPS) {
            float s2 = 0.f;
            for (int i = lane; i < per; i += 32) { const float v = xs[g * per + i]; s2 = fmaf(v, v, s2); }
            s2 = warp_sum(s2);
            if (lane == 0) inv_g[g] = 1.0f / sqrtf(s2 / (float)per + eps);
        }
        __syncthreads();
        for (int i = threadIdx.x; i < K; i += DV_WARPS * 32) xs[i] = xs[i] * inv_g[i / per] * norm_w[i];
    } else if (norm_w) {
        // RMS norm of the staged vector: every CTA sums the squares in the same order, so all CTAs (and every launch that reads the
        // same x) derive the bit-identical normalised vector
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xFFFFFFFFu, ss, o);
        if (lane == 0) red[warp] = ss;
        __syncthreads();
        float tot = 0.f;
#pragma unroll
        for (int w = 0; w < DV_WARPS; w++) tot += red[w];
        const float inv = 1.0f / sqrtf(tot / (float)K + eps);
        for (int i = threadIdx.x; i < K; i += DV_WARPS * 32) xs[i] = xs[i] * inv * norm_w[i];
    }
    __syncthreads();
    const bool glu = ep == DENSE_SWIGLU || ep == DENSE_GEGLU || ep == DENSE_REGLU;
    int total = m.out[0];
    if (!glu) for (int i = 1; i < m.n; i++) total += m.out[i];
    for (int r = blockIdx.x * DV_WARPS + warp; r < total; r += gridDim.x * DV_WARPS) {
        if (glu) {
            const float g = dense_row_dot<T>(m.W[0] + (size_t)r * m.pitch[0], xs, K, lane, vec);
            const float u = dense_row_dot<T>(m.W[1] + (size_t)r * m.pitch[1], xs, K, lane, vec);
            if (lane == 0) m.y[0][r] = (ep == DENSE_GEGLU ? gelu_tanh_f(g) : ep == DENSE_REGLU ? fmaxf(g, 0.f) : silu_f(g)) * u;
            continue;
        }
        int mi = 0, row = r;
        while (mi + 1 < m.n && row >= m.out[mi]) { row -= m.out[mi]; mi++; }
        const float v = dense_row_dot<T>(m.W[mi] + (size_t)row * m.pitch[mi], xs, K, lane, vec);
        if (lane == 0 && ep == DENSE_STREAMS) streams_update(sio, m.out[0], row, v);
        else if (lane == 0) {
            float* y = m.y[mi] + row;
            if (ep == DENSE_ADD) *y += v;
            else if (ep == DENSE_SCALED_ADD) *y = fmaf(alpha * (row_scale ? row_scale[row] : 1.f), v, *y);
            else *y = v;
        }
    }
}

// n floats into shared memory by the whole CTA, 16 bytes at a time when the source is aligned.  planar (n % 8 == 0): the even and the odd
// 16-byte pieces go to the first and the second half of dst, so that lanes holding consecutive 8-number pieces of a 16-bit weight row read
// consecutive 16-byte words of either half (no bank conflicts).
__device__ __forceinline__ void stage_floats(float* dst, const float* src, int n, bool planar) {
    const bool al = (reinterpret_cast<uintptr_t>(src) & 15) == 0;
    if (planar) {
        const int half = n >> 1, q = n >> 2;
        if (al) {
#pragma unroll 4
            for (int i = threadIdx.x; i < q; i += blockDim.x) *reinterpret_cast<float4*>(dst + ((i & 1) ? half : 0) + (i >> 1) * 4) = *reinterpret_cast<const float4*>(src + 4 * i);
        } else {
            for (int i = threadIdx.x; i < n; i += blockDim.x) dst[((i & 4) ? half : 0) + (i >> 3) * 4 + (i & 3)] = src[i];
        }
        return;
    }
    int done = 0;
    if (al) {
        done = n & ~3;
#pragma unroll 4
        for (int i = threadIdx.x * 4; i < done; i += blockDim.x * 4) *reinterpret_cast<float4*>(dst + i) = *reinterpret_cast<const float4*>(src + i);
    }
    for (int i = done + threadIdx.x; i < n; i += blockDim.x) dst[i] = src[i];
}
// acc += <the 16-byte weight piece w, its numbers of the staged vector>; v: the piece's index in the row of K numbers
template <typename T>
__device__ __forceinline__ float piece_dot(const uint4& w, const float* xs, int K, int v, float acc) {
    constexpr int P = Elem<T>::PER16;
    float f[P];
    Elem<T>::unpack(w, f);
    const float4 a = *reinterpret_cast<const float4*>(xs + 4 * v);
    acc = fmaf(f[0], a.x, acc); acc = fmaf(f[1], a.y, acc); acc = fmaf(f[2], a.z, acc); acc = fmaf(f[3], a.w, acc);
    if constexpr (P == 8) {
        const float4 b = *reinterpret_cast<const float4*>(xs + (K >> 1) + 4 * v);
        acc = fmaf(f[4], b.x, acc); acc = fmaf(f[5], b.y, acc); acc = fmaf(f[6], b.z, acc); acc = fmaf(f[7], b.w, acc);
    }
    return acc;
}
// batch of up to 128 pieces from v0 on, four 16-byte loads in flight per lane
template <typename T>
__device__ __forceinline__ float batch_dot(const unsigned char* row, const float* xs, int K, int nv, int v0, int lane, float acc) {
    uint4 w[4];
#pragma unroll
    for (int u = 0; u < 4; u++) { const int v = v0 + lane + 32 * u; w[u] = v < nv ? ld_stream16(row + (size_t)v * 16) : make_uint4(0u, 0u, 0u, 0u); }
#pragma unroll
    for (int u = 0; u < 4; u++) acc = piece_dot<T>(w[u], xs, K, min(v0 + lane + 32 * u, nv - 1), acc);       // past the end the weights are zeros: any valid input will do
    return acc;
}

// ---- several matrices, each with its own input vector ----
struct MultiDev {
    struct One { const unsigned char* W; size_t pitch; const float* x; float* y; const float* act_p; const float* norm_w; float eps; int out, K, act, f32, vec, cta_end; };
    One m[DENSE_MAX_MATS];
    int n;
};
// A CTA serves rows of one matrix: it stages that matrix's input, then a warp per row.
template <typename T>
__global__ void __launch_bounds__(DV_WARPS * 32) gemv_multi_kernel(const __grid_constant__ MultiDev md) {
    extern __shared__ __align__(16) float xs[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    int mi = 0, first = 0;
    while (mi + 1 < md.n && (int)blockIdx.x >= md.m[mi].cta_end) { first = md.m[mi].cta_end; mi++; }
    const MultiDev::One& m = md.m[mi];
    const int ctas = m.cta_end - first, r0 = ((int)blockIdx.x - first) * DV_WARPS + warp;
    const size_t row_bytes = (size_t)m.K * (m.f32 ? sizeof(float) : sizeof(T));
    for (int r = r0; r < m.out; r += ctas * DV_WARPS) l2_prefetch(m.W + (size_t)r * m.pitch, row_bytes, lane, 32);
    pdl_wait();
    const bool wide = !m.f32 && m.vec;                    // 16-bit rows in whole pieces: planar staging
    float inv = 1.f;
    if (m.norm_w) {                                       // the gain goes into the staged vector, the root mean square onto the results
        __shared__ float red[DV_WARPS];
        const bool planar = wide && Elem<T>::PER16 == 8;
        const int half = m.K >> 1;
        float ss = 0.f;
        for (int i = threadIdx.x; i < m.K; i += DV_WARPS * 32) {
            const float v = m.x[i];
            ss = fmaf(v, v, ss);
            xs[planar ? ((i & 4) ? half : 0) + (i >> 3) * 4 + (i & 3) : i] = v * m.norm_w[i];
        }
        ss = warp_sum(ss);
        if (lane == 0) red[warp] = ss;
        __syncthreads();
        float tot = 0.f;
#pragma unroll
        for (int w = 0; w < DV_WARPS; w++) tot += red[w];
        inv = 1.0f / sqrtf(tot / (float)m.K + m.eps);
    } else stage_floats(xs, m.x, m.K, wide && Elem<T>::PER16 == 8);
    __syncthreads();
    float a = 0.f, b = 0.f;
    if (m.act == GEMV_ACT_XIELU) { a = softplus_f(m.act_p[0]); b = softplus_f(m.act_p[1]); }
    for (int r = r0; r < m.out; r += ctas * DV_WARPS) {
        const unsigned char* row = m.W + (size_t)r * m.pitch;
        float v = 0.f;
        if (wide) {
            const int nv = m.K / Elem<T>::PER16;
            for (int v0 = 0; v0 < nv; v0 += 128) v = batch_dot<T>(row, xs, m.K, nv, v0, lane, v);
            v = warp_sum(v);
        } else v = m.f32 ? dense_row_dot<float>(row, xs, m.K, lane, m.vec) : dense_row_dot<T>(row, xs, m.K, lane, m.vec);
        if (lane == 0) {
            v *= inv;
            if (m.act == GEMV_ACT_TANH) v = tanhf(v);
            else if (m.act == GEMV_ACT_XIELU) v = xielu_f(v, a, b);
            else if (m.act == GEMV_ACT_RELU2) { v = fmaxf(v, 0.f); v *= v; }
            m.y[r] = v;
        }
    }
    pdl_launch_dependents();       // late: CTAs of a small dependent grid placed while this one fills the SMs would crowd onto the few that free up first
}

// ---- y[r] (+)= sum over terms of <W[r], x> (routed term: sum_k wt[k] <table[sel[k]][r], x_k>) ----
struct SumDev {
    struct One { const unsigned char* W; const void* const* table; const int* sel; const float* wt; const float* x; int K, top, vec, at; };
    One t[GEMV_SUM_MAX_TERMS];
    int n, out, add, nw;
    float* y;
};
// A CTA of SV_WARPS warps owns SV_WARPS / nw rows at a time, nw warps per row: the batches of 128 16-byte pieces of a row's terms (of all terms,
// one count) go round the row's warps; their sums meet in shared memory in a fixed order.
constexpr int SV_WARPS = 16;
template <typename T>
__device__ __forceinline__ float row_batches(const unsigned char* row, const float* xs, int K, int lane, bool vec, int& count, int j, int nw) {
    constexpr int P = Elem<T>::PER16;
    float acc = 0.f;
    if (vec) {
        const int nv = K / P;
        for (int v0 = 0; v0 < nv; v0 += 128) {
            if (count++ % nw != j) continue;
            acc = batch_dot<T>(row, xs, K, nv, v0, lane, acc);
        }
    } else {
        for (int i0 = 0; i0 < K; i0 += 1024) {
            if (count++ % nw != j) continue;
            for (int i = i0 + lane; i < min(K, i0 + 1024); i += 32) acc = fmaf(Elem<T>::one(row, i), xs[i], acc);
        }
    }
    return acc;
}
template <typename T>
__global__ void __launch_bounds__(SV_WARPS * 32) gemv_sum_kernel(const __grid_constant__ SumDev sd) {
    extern __shared__ __align__(16) float xs[];
    __shared__ float part[SV_WARPS];
    __shared__ const unsigned char* routed[256];       // the chosen experts' matrices and weights of a routed term
    __shared__ float routed_w[256];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = sd.nw, rows = SV_WARPS / nw, j = warp % nw, rl = warp / nw;
    for (int r = blockIdx.x * rows + rl; r < sd.out; r += gridDim.x * rows)
        for (int q = 0; q < sd.n; q++)
            if (!sd.t[q].table) l2_prefetch(sd.t[q].W + (size_t)r * sd.t[q].K * sizeof(T), (size_t)sd.t[q].K * sizeof(T), lane + 32 * j, 32 * nw);
    pdl_wait();
    for (int q = 0; q < sd.n; q++)
        if (sd.t[q].table)
            for (int k = threadIdx.x; k < sd.t[q].top; k += SV_WARPS * 32) { routed[k] = static_cast<const unsigned char*>(sd.t[q].table[sd.t[q].sel[k]]); routed_w[k] = sd.t[q].wt[k]; }
    for (int q = 0; q < sd.n; q++)
        for (int k = 0; k < sd.t[q].top; k++) stage_floats(xs + sd.t[q].at + k * sd.t[q].K, sd.t[q].x + (size_t)k * sd.t[q].K, sd.t[q].K, sd.t[q].vec && Elem<T>::PER16 == 8);
    __syncthreads();
    for (int base = blockIdx.x * rows; base < sd.out; base += gridDim.x * rows) {
        const int r = base + rl;
        float acc = 0.f;
        if (r < sd.out) {
            int count = 0;
            for (int q = 0; q < sd.n; q++) {
                const SumDev::One& t = sd.t[q];
                const size_t off = (size_t)r * t.K * sizeof(T);
                if (!t.table) acc += row_batches<T>(t.W + off, xs + t.at, t.K, lane, t.vec, count, j, nw);
                else for (int k = 0; k < t.top; k++)
                    acc = fmaf(routed_w[k], row_batches<T>(routed[k] + off, xs + t.at + k * t.K, t.K, lane, t.vec, count, j, nw), acc);
            }
        }
        acc = warp_sum(acc);
        if (lane == 0) part[warp] = acc;
        __syncthreads();
        if (threadIdx.x < rows && base + (int)threadIdx.x < sd.out) {
            float v = 0.f;
            for (int w = 0; w < nw; w++) v += part[threadIdx.x * nw + w];
            float* y = sd.y + base + threadIdx.x;
            *y = sd.add ? *y + v : v;
        }
        __syncthreads();
    }
    pdl_launch_dependents();
}

template <bool VEC>
__global__ void __launch_bounds__(256) xielu_kernel(float* __restrict__ out, __nv_bfloat16* __restrict__ hi, size_t lo, const float* __restrict__ in, const float* __restrict__ act_p, size_t n) {
    pdl_launch_dependents();
    pdl_wait();
    constexpr int V = VEC ? 4 : 1;
    const size_t i = ((size_t)blockIdx.x * 256 + threadIdx.x) * V;
    if (i >= n) return;
    const float a = softplus_f(act_p[0]), b = softplus_f(act_p[1]);
    float v[V];
    if constexpr (VEC) { const float4 f = *reinterpret_cast<const float4*>(in + i); v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w; } else v[0] = in[i];
#pragma unroll
    for (int e = 0; e < V; e++) v[e] = xielu_f(v[e], a, b);
    if (out) { if constexpr (VEC) *reinterpret_cast<float4*>(out + i) = make_float4(v[0], v[1], v[2], v[3]); else out[i] = v[0]; }
    if (hi) { if constexpr (VEC) split_store4(hi, hi + lo, i, v); else split_store1(hi, hi + lo, i, v[0]); }
}

// ---- C[T,N] (ep)= A[T,K] . W[N,K]^T on CUDA cores ----
constexpr int GT = 64, GK = 16;
template <typename T>
__global__ void __launch_bounds__(256) gemm_dense_kernel(float* __restrict__ C, const float* __restrict__ A, const unsigned char* __restrict__ W,
                                                         size_t pitch, int Tn, int N, int K, int ep, const float* __restrict__ row_scale, float alpha) {
    __shared__ float As[GK][GT + 4];
    __shared__ float Ws[GK][GT + 4];
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    const int t0 = blockIdx.y * GT, n0 = blockIdx.x * GT;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < K; k0 += GK) {
        for (int e = threadIdx.x; e < GT * GK; e += 256) {
            const int r = e / GK, k = e % GK;
            const int t = t0 + r, n = n0 + r, kk = k0 + k;
            As[k][r] = (t < Tn && kk < K) ? A[(size_t)t * K + kk] : 0.f;
            Ws[k][r] = (n < N && kk < K) ? Elem<T>::one(W + (size_t)n * pitch, kk) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < GK; k++) {
            float a[4], w[4];
#pragma unroll
            for (int i = 0; i < 4; i++) { a[i] = As[k][ty * 4 + i]; w[i] = Ws[k][tx * 4 + i]; }
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(a[i], w[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const int t = t0 + ty * 4 + i;
        if (t >= Tn) continue;
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int n = n0 + tx * 4 + j;
            if (n >= N) continue;
            float* c = C + (size_t)t * N + n;
            if (ep == DENSE_ADD) *c += acc[i][j];
            else if (ep == DENSE_SCALED_ADD) *c = fmaf(alpha * (row_scale ? row_scale[n] : 1.f), acc[i][j], *c);
            else *c = acc[i][j];
        }
    }
}

__global__ void glu_mul_kernel(float* __restrict__ out, const float* __restrict__ gate, const float* __restrict__ up, size_t n, int act) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) out[i] = (act == 1 ? gelu_tanh_f(gate[i]) : act == 2 ? fmaxf(gate[i], 0.f) : silu_f(gate[i])) * up[i];
}
__global__ void scaled_add_rows_kernel(float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ row_scale, float alpha,
                                       size_t n, int cols) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) x[i] = fmaf(alpha * (row_scale ? row_scale[i % cols] : 1.f), y[i], x[i]);
}
__global__ void copy_cols_kernel(float* __restrict__ out, const float* __restrict__ in, size_t n, int cols, int ld) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) out[i] = in[(i / cols) * ld + i % cols];
}
template <typename T>
__global__ void to_f32_kernel(float* __restrict__ out, const T* __restrict__ in, size_t n) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) out[i] = Elem<T>::one(in + i, 0);
}

}  // namespace

bool dense_dtype(DType dt) { return dt == DType::F32 || dt == DType::F16 || dt == DType::BF16; }

void gemv_dense(const GemvMat* mats, int n_mat, int K, const float* x, DenseEpilogue ep, const float* row_scale, float alpha, cudaStream_t s,
                const float* norm_w, float eps, const StreamsIO* sio_p, int norm_groups) {
    NT_CHECK(norm_groups >= 1 && norm_groups <= DENSE_MAX_NORM_GROUPS && K % norm_groups == 0, "gemv_dense: norm groups must be equal parts, at most 256");
    NT_CHECK(n_mat >= 1 && n_mat <= DENSE_MAX_MATS, "gemv_dense: too many matrices for one launch");
    const StreamsIO sio = sio_p ? *sio_p : StreamsIO();
    NT_CHECK(ep != DENSE_STREAMS || (n_mat == 1 && sio.X_out && sio.M && sio.b && sio.S >= 1 && sio.S <= 16), "gemv_dense: the streams epilogue takes one matrix and the stream tables");
    NT_CHECK(!sio.X_in || (sio.S >= 1 && sio.S <= 16), "gemv_dense: 1..16 streams");
    const bool glu = ep == DENSE_SWIGLU || ep == DENSE_GEGLU || ep == DENSE_REGLU;
    NT_CHECK(!glu || (n_mat == 2 && mats[0].out == mats[1].out), "gemv_dense: a gated epilogue takes two matrices of equal height");
    const DType dt = mats[0].dtype;
    NT_CHECK(dense_dtype(dt), "gemv_dense: dense dtypes only");
    DenseMats m{};
    m.n = n_mat;
    const int per16 = dt == DType::F32 ? 4 : 8;
    int vec = (K % per16 == 0) ? 1 : 0, total = 0;
    for (int i = 0; i < n_mat; i++) {
        NT_CHECK(mats[i].dtype == dt, "gemv_dense: one dtype per launch");
        m.W[i] = static_cast<const unsigned char*>(mats[i].W); m.y[i] = mats[i].y; m.out[i] = mats[i].out;
        m.pitch[i] = mats[i].row_pitch ? mats[i].row_pitch : dtype_row_size(dt, (size_t)K);
        if ((reinterpret_cast<uintptr_t>(mats[i].W) & 15) || (m.pitch[i] & 15)) vec = 0;
        total += mats[i].out;
    }
    if (glu) total = mats[0].out;
    if (total <= 0) return;
    const size_t smem = (size_t)K * sizeof(float);
    NT_CHECK(smem <= 200 * 1024, "gemv_dense: the activation vector does not fit in shared memory");
    int grid = (total + DV_WARPS - 1) / DV_WARPS;
    const int resident = (int)std::max<size_t>(1, std::min<size_t>(8, (size_t)(220 * 1024) / (smem + 1024))) * 148;
    grid = std::min(grid, resident);
#define NT_DV(TY) { static unsigned long long done = 0; if (smem > 40 * 1024) opt_in_dynamic_smem(gemv_dense_kernel<TY>, 200 * 1024, done); \
                    launch_k(gemv_dense_kernel<TY>, dim3(grid), dim3(DV_WARPS * 32), smem, s, m, x, K, (int)ep, row_scale, alpha, vec, norm_w, eps, sio, norm_groups); }
    if (dt == DType::F32) NT_DV(float) else if (dt == DType::F16) NT_DV(__half) else NT_DV(__nv_bfloat16)
#undef NT_DV
    count_launch();
}

void gemv_multi(const MultiMat* mats, int n_mat, cudaStream_t s) {
    NT_CHECK(n_mat >= 1 && n_mat <= DENSE_MAX_MATS, "gemv_multi: too many matrices for one launch");
    MultiDev md{};
    md.n = n_mat;
    DType dt = DType::F32;
    for (int i = 0; i < n_mat; i++) if (mats[i].dtype != DType::F32) dt = mats[i].dtype;
    size_t bytes[DENSE_MAX_MATS], total = 0;
    int K = 0, rows = 0;
    for (int i = 0; i < n_mat; i++) {
        const MultiMat& a = mats[i];
        NT_CHECK(dense_dtype(a.dtype) && (a.dtype == dt || a.dtype == DType::F32), "gemv_multi: one 16-bit dtype per launch (beside F32 tables)");
        NT_CHECK(a.act != GEMV_ACT_XIELU || a.act_p, "gemv_multi: the activation's two numbers are missing");
        MultiDev::One& o = md.m[i];
        o.W = static_cast<const unsigned char*>(a.W); o.pitch = a.row_pitch ? a.row_pitch : dtype_row_size(a.dtype, (size_t)a.K);
        o.x = a.x; o.y = a.y; o.act_p = a.act_p; o.norm_w = a.norm_w; o.eps = a.eps; o.out = a.out; o.K = a.K; o.act = a.act; o.f32 = a.dtype == DType::F32 ? 1 : 0;
        o.vec = a.K % (o.f32 ? 4 : 8) == 0 && (reinterpret_cast<uintptr_t>(a.W) & 15) == 0 && (o.pitch & 15) == 0;
        bytes[i] = (size_t)a.out * o.pitch; total += bytes[i];
        K = std::max(K, a.K); rows += a.out;
    }
    if (rows <= 0) return;
    const size_t smem = (size_t)K * sizeof(float);
    NT_CHECK(smem <= 200 * 1024, "gemv_multi: the activation vector does not fit in shared memory");
    // CTAs by share of the bytes, no more than resident at once: a warp's rows follow each other without a second wave
    const int resident = (int)std::max<size_t>(1, std::min<size_t>(8, (size_t)(220 * 1024) / (smem + 1024))) * 148;
    int end = 0;
    for (int i = 0; i < n_mat; i++) {
        const int full = (mats[i].out + DV_WARPS - 1) / DV_WARPS;
        const int share = (int)((double)resident * (double)bytes[i] / (double)std::max<size_t>(1, total));
        end += std::max(1, std::min(full, share));
        md.m[i].cta_end = end;
    }
#define NT_MV(TY) { static unsigned long long done = 0; if (smem > 40 * 1024) opt_in_dynamic_smem(gemv_multi_kernel<TY>, 200 * 1024, done); \
                    launch_k(gemv_multi_kernel<TY>, dim3(end), dim3(DV_WARPS * 32), smem, s, md); }
    if (dt == DType::F32) NT_MV(float) else if (dt == DType::F16) NT_MV(__half) else NT_MV(__nv_bfloat16)
#undef NT_MV
    count_launch();
}

void gemv_sum(float* y, const SumTerm* terms, int n, int out, DType dt, bool add, cudaStream_t s) {
    NT_CHECK(n >= 1 && n <= GEMV_SUM_MAX_TERMS && dense_dtype(dt), "gemv_sum: 1..4 terms of a dense dtype");
    if (out <= 0) return;
    SumDev sd{};
    sd.n = n; sd.out = out; sd.add = add ? 1 : 0; sd.y = y;
    int at = 0;
    int n_routed = 0;
    for (int i = 0; i < n; i++) {
        const SumTerm& t = terms[i];
        if (t.table) n_routed++;
        NT_CHECK(!t.table || (n_routed == 1 && t.top >= 1 && t.top <= 256), "gemv_sum: one routed term of at most 256 chosen matrices");
        SumDev::One& o = sd.t[i];
        o.W = static_cast<const unsigned char*>(t.W); o.table = t.table; o.sel = t.sel; o.wt = t.wt; o.x = t.x; o.K = t.K; o.top = t.table ? t.top : 1; o.at = at;
        o.vec = t.K % (dt == DType::F32 ? 4 : 8) == 0 && (t.table ? t.table_aligned : (reinterpret_cast<uintptr_t>(t.W) & 15) == 0);
        at += (t.K * o.top + 3) & ~3;
    }
    const size_t smem = (size_t)at * sizeof(float);
    NT_CHECK(smem <= 200 * 1024, "gemv_sum: the input vectors do not fit in shared memory");
    // warps per row: as many as keep the grid within what is resident at once (64 warps per SM)
    const int per_sm = (int)std::max<size_t>(1, std::min<size_t>(4, (size_t)(220 * 1024) / (smem + 1024)));
    sd.nw = 1;
    while (sd.nw < 4 && (long)out * sd.nw * 2 <= (long)148 * per_sm * SV_WARPS) sd.nw *= 2;
    const int rows = SV_WARPS / sd.nw, grid = std::min((out + rows - 1) / rows, 148 * per_sm);
#define NT_SV(TY) { static unsigned long long done = 0; if (smem > 40 * 1024) opt_in_dynamic_smem(gemv_sum_kernel<TY>, 200 * 1024, done); \
                    launch_k(gemv_sum_kernel<TY>, dim3(grid), dim3(SV_WARPS * 32), smem, s, sd); }
    if (dt == DType::F32) NT_SV(float) else if (dt == DType::F16) NT_SV(__half) else NT_SV(__nv_bfloat16)
#undef NT_SV
    count_launch();
}

void xielu_rows(float* out, void* split, const float* in, const float* act_p, int T, int cols, cudaStream_t s) {
    const size_t n = (size_t)T * cols;
    if (!n) return;
    const bool vec = n % 4 == 0 && cols % 4 == 0 && ((reinterpret_cast<uintptr_t>(in) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(split)) & 15) == 0;
    const dim3 grid((unsigned)((n + (vec ? 1023 : 255)) / (vec ? 1024 : 256)));
    __nv_bfloat16* hi = static_cast<__nv_bfloat16*>(split);
    if (vec) launch_k(xielu_kernel<true>, grid, dim3(256), 0, s, out, hi, split_lo_offset(T, cols), in, act_p, n);
    else launch_k(xielu_kernel<false>, grid, dim3(256), 0, s, out, hi, split_lo_offset(T, cols), in, act_p, n);
    count_launch();
}

void gemm_dense(float* C, const float* A, const void* W, DType dt, size_t row_pitch, int T, int N, int K, DenseEpilogue ep,
                const float* row_scale, float alpha, cudaStream_t s) {
    NT_CHECK(dense_dtype(dt), "gemm_dense: dense dtypes only");
    NT_CHECK(ep == DENSE_STORE || ep == DENSE_ADD || ep == DENSE_SCALED_ADD, "gemm_dense: store / add / scaled-add epilogues");
    if (T <= 0 || N <= 0) return;
    const size_t pitch = row_pitch ? row_pitch : dtype_row_size(dt, (size_t)K);
    const dim3 grid((N + GT - 1) / GT, (T + GT - 1) / GT);
    const unsigned char* w = static_cast<const unsigned char*>(W);
    if (dt == DType::F32) gemm_dense_kernel<float><<<grid, 256, 0, s>>>(C, A, w, pitch, T, N, K, (int)ep, row_scale, alpha);
    else if (dt == DType::F16) gemm_dense_kernel<__half><<<grid, 256, 0, s>>>(C, A, w, pitch, T, N, K, (int)ep, row_scale, alpha);
    else gemm_dense_kernel<__nv_bfloat16><<<grid, 256, 0, s>>>(C, A, w, pitch, T, N, K, (int)ep, row_scale, alpha);
    NT_LAUNCH_CHECK();
    count_launch();
}

void glu_mul(float* out, const float* gate, const float* up, size_t n, bool gelu, cudaStream_t s, bool relu) {
    if (!n) return;
    glu_mul_kernel<<<(unsigned)((n + 255) / 256), 256, 0, s>>>(out, gate, up, n, relu ? 2 : (gelu ? 1 : 0));
    NT_LAUNCH_CHECK();
    count_launch();
}

void copy_cols(float* out, const float* in, int rows, int cols, int ld, cudaStream_t s) {
    const size_t n = (size_t)rows * cols;
    if (!n) return;
    copy_cols_kernel<<<(unsigned)((n + 255) / 256), 256, 0, s>>>(out, in, n, cols, ld);
    NT_LAUNCH_CHECK();
    count_launch();
}

void scaled_add_rows(float* x, const float* y, const float* row_scale, float alpha, int rows, int cols, cudaStream_t s) {
    const size_t n = (size_t)rows * cols;
    if (!n) return;
    scaled_add_rows_kernel<<<(unsigned)((n + 255) / 256), 256, 0, s>>>(x, y, row_scale, alpha, n, cols);
    NT_LAUNCH_CHECK();
    count_launch();
}

void dense_to_f32(float* out, const void* in, DType dt, size_t n, cudaStream_t s) {
    if (!n) return;
    const unsigned g = (unsigned)((n + 255) / 256);
    if (dt == DType::F32) NT_CUDA_CHECK(cudaMemcpyAsync(out, in, n * 4, cudaMemcpyDeviceToDevice, s));
    else if (dt == DType::F16) to_f32_kernel<__half><<<g, 256, 0, s>>>(out, static_cast<const __half*>(in), n);
    else if (dt == DType::BF16) to_f32_kernel<__nv_bfloat16><<<g, 256, 0, s>>>(out, static_cast<const __nv_bfloat16*>(in), n);
    else NT_CHECK(false, "dense_to_f32: dense dtypes only");
    NT_LAUNCH_CHECK();
}

}}  // namespace nt::b200
