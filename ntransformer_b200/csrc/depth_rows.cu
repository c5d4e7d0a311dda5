// depth_rows.cu — row-wise pieces around the layers of a model whose layer inputs are averages over the depth (ModelConfig::depth_average)
// and whose norms work on groups of channels (ModelConfig::norm_groups), all F32:
//   embed_bigram_rows   X_0[t] = E[token_t] + B[(token_{t-1} * mul_prev + token_t * mul_cur) mod buckets]; a sequence's first token reads
//                       row `buckets` of B.  The token before the step's first row is sequence state (one int on the device).
//   depth_norm_rows     x = sum_j c_j X_j over the slots X_0 .. X_{n-1} (c == null: the last slot alone), stored as the base the next
//                       layer's branches are added to; h = x / rms(its group) * gain, as F32 rows and / or as the BF16 split the
//                       tensor-core GEMM reads.  One decoded token can also take the token-shift blends h + (h' - h) mu_s of the
//                       next mixer from the same pass (h' the previous token's h, sequence state, replaced here).
//                       One CTA per (row, group): the groups of a row are independent.
// A step's base position is *pos_dev when given (the captured decode step), else p0.  Compiled WITHOUT --use_fast_math.
#include "kernels_internal.h"
#include "bf16_split.cuh"
#include "ring.cuh"
#include <cuda_fp16.h>
#include <algorithm>

namespace nt { namespace b200 {

namespace {

__device__ __forceinline__ float eld(const void* p, int dt, size_t i) {
    if (dt == (int)DType::F32) return static_cast<const float*>(p)[i];
    if (dt == (int)DType::F16) return __half2float(static_cast<const __half*>(p)[i]);
    return __bfloat162float(static_cast<const __nv_bfloat16*>(p)[i]);
}

__global__ void __launch_bounds__(256) embed_bigram_kernel(float* __restrict__ x0, float* __restrict__ x1, const void* __restrict__ E, int edt, const void* __restrict__ B,
                                                           int bdt, const int* __restrict__ tokens, const int* __restrict__ prev, int width, long long buckets,
                                                           long long mul_prev, long long mul_cur, const int* __restrict__ pos_dev, int p0) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.y, i = blockIdx.x * 256 + threadIdx.x;
    if (i >= width) return;
    const long long tok = tokens[t];
    float v = eld(E, edt, (size_t)tok * width + i);
    if (B) {
        const bool first = t == 0 && (pos_dev ? *pos_dev : p0) == 0;
        long long row = buckets;
        if (!first) {
            const long long before = t > 0 ? tokens[t - 1] : *prev;
            row = (before * mul_prev + tok * mul_cur) % buckets;
            if (row < 0) row += buckets;
        }
        v += eld(B, bdt, (size_t)row * width + i);
    }
    x0[(size_t)t * width + i] = v;
    if (x1) x1[(size_t)t * width + i] = v;
}

template <int VEC> struct Pack { float v[VEC]; };
template <int VEC> __device__ __forceinline__ Pack<VEC> ldp(const float* p);
template <> __device__ __forceinline__ Pack<1> ldp<1>(const float* p) { Pack<1> r; r.v[0] = *p; return r; }
template <> __device__ __forceinline__ Pack<4> ldp<4>(const float* p) { const float4 f = *reinterpret_cast<const float4*>(p); Pack<4> r; r.v[0] = f.x; r.v[1] = f.y; r.v[2] = f.z; r.v[3] = f.w; return r; }
__device__ __forceinline__ void stp(float* p, const Pack<1>& a) { *p = a.v[0]; }
__device__ __forceinline__ void stp(float* p, const Pack<4>& a) { *reinterpret_cast<float4*>(p) = make_float4(a.v[0], a.v[1], a.v[2], a.v[3]); }

constexpr int DN_KEEP = 4;       // packs of a thread that stay in registers between the two passes; further ones are summed again

template <int VEC>
__global__ void __launch_bounds__(256) depth_norm_kernel(DepthNorm p) {
    __shared__ float red[8];
    const int per = p.width / p.groups, c0 = blockIdx.y * per, n = per / VEC, nt = blockDim.x;
    if (p.n_mix > 0) {
        l2_prefetch(p.gain + c0, (size_t)per * sizeof(float), threadIdx.x, nt);
        for (int s = 0; s < p.n_mix; s++) l2_prefetch(p.mu[s] + c0, (size_t)per * sizeof(float), threadIdx.x, nt);
    }
    pdl_launch_dependents();
    pdl_wait();
    const size_t row = (size_t)blockIdx.x * p.width + c0;
    auto blend = [&](int i) {
        Pack<VEC> a;
        const float* x = p.X + row + (size_t)i * VEC;
        if (!p.coef) return ldp<VEC>(x + (size_t)(p.n - 1) * p.slot);
#pragma unroll
        for (int e = 0; e < VEC; e++) a.v[e] = 0.f;
#pragma unroll 4
        for (int j = 0; j < p.n; j++) {
            const Pack<VEC> v = ldp<VEC>(x + (size_t)j * p.slot);
            const float c = __ldg(p.coef + j);
#pragma unroll
            for (int e = 0; e < VEC; e++) a.v[e] = fmaf(c, v.v[e], a.v[e]);
        }
        return a;
    };
    Pack<VEC> keep[DN_KEEP];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < DN_KEEP; k++) {
        const int i = threadIdx.x + k * nt;
        if (i < n) {
            keep[k] = blend(i);
#pragma unroll
            for (int e = 0; e < VEC; e++) ss = fmaf(keep[k].v[e], keep[k].v[e], ss);
            if (p.x_out) stp(p.x_out + row + (size_t)i * VEC, keep[k]);
        }
    }
    for (int i = threadIdx.x + DN_KEEP * nt; i < n; i += nt) {
        const Pack<VEC> a = blend(i);
#pragma unroll
        for (int e = 0; e < VEC; e++) ss = fmaf(a.v[e], a.v[e], ss);
        if (p.x_out) stp(p.x_out + row + (size_t)i * VEC, a);
    }
    if (!p.gain) return;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xFFFFFFFFu, ss, o);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    float tot = 0.f;
    for (int w = 0; w < (nt >> 5); w++) tot += red[w];
    const float inv = 1.0f / sqrtf(tot / (float)per + p.eps);
    const bool fresh = p.n_mix > 0 && (p.pos_dev ? *p.pos_dev : p.p0) == 0;
    auto emit = [&](int i, const Pack<VEC>& a) {
        const size_t c = (size_t)c0 + (size_t)i * VEC;
        const Pack<VEC> g = ldp<VEC>(p.gain + c);
        Pack<VEC> h;
#pragma unroll
        for (int e = 0; e < VEC; e++) h.v[e] = a.v[e] * inv * g.v[e];
        const size_t at = row + (size_t)i * VEC;
        if (p.h_out) stp(p.h_out + at, h);
        if (p.split) {
            __nv_bfloat16* hi = static_cast<__nv_bfloat16*>(p.split);
            if constexpr (VEC == 4) split_store4(hi, hi + p.split_lo, at, h.v);
            else split_store1(hi, hi + p.split_lo, at, h.v[0]);
        }
        if (p.n_mix > 0) {                                  // one row: the previous token's h is the carried row
            Pack<VEC> prev;
#pragma unroll
            for (int e = 0; e < VEC; e++) prev.v[e] = 0.f;
            if (!fresh) prev = ldp<VEC>(p.carried + c);
            for (int s = 0; s < p.n_mix; s++) {
                const Pack<VEC> mu = ldp<VEC>(p.mu[s] + c);
                Pack<VEC> m;
#pragma unroll
                for (int e = 0; e < VEC; e++) m.v[e] = fmaf(prev.v[e] - h.v[e], mu.v[e], h.v[e]);
                stp(p.mix_out[s] + c, m);
            }
            stp(p.carried + c, h);
        }
    };
#pragma unroll
    for (int k = 0; k < DN_KEEP; k++) { const int i = threadIdx.x + k * nt; if (i < n) emit(i, keep[k]); }
    for (int i = threadIdx.x + DN_KEEP * nt; i < n; i += nt) emit(i, blend(i));
}

// The same over prompt rows for groups of at most 32 * DN_KEEP 16-byte pieces: a warp per (row, group), no barrier.
__global__ void __launch_bounds__(256) depth_norm_warp_kernel(DepthNorm p, int n_items) {
    pdl_launch_dependents();
    pdl_wait();
    const int item = (int)blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (item >= n_items) return;
    const int per = p.width / p.groups, n = per / 4, t = item / p.groups, c0 = (item - t * p.groups) * per;
    const size_t row = (size_t)t * p.width + c0;
    Pack<4> keep[DN_KEEP];
#pragma unroll
    for (int k = 0; k < DN_KEEP; k++)
#pragma unroll
        for (int e = 0; e < 4; e++) keep[k].v[e] = 0.f;
    for (int j = p.coef ? 0 : p.n - 1; j < p.n; j++) {
        const float c = p.coef ? __ldg(p.coef + j) : 1.f;
        const float* x = p.X + (size_t)j * p.slot + row;
#pragma unroll
        for (int k = 0; k < DN_KEEP; k++) {
            const int i = lane + 32 * k;
            if (i < n) {
                const Pack<4> v = ldp<4>(x + 4 * i);
#pragma unroll
                for (int e = 0; e < 4; e++) keep[k].v[e] = fmaf(c, v.v[e], keep[k].v[e]);
            }
        }
    }
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < DN_KEEP; k++) {
        const int i = lane + 32 * k;
        if (i < n) {
#pragma unroll
            for (int e = 0; e < 4; e++) ss = fmaf(keep[k].v[e], keep[k].v[e], ss);
            if (p.x_out) stp(p.x_out + row + 4 * (size_t)i, keep[k]);
        }
    }
    if (!p.gain) return;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xFFFFFFFFu, ss, o);
    const float inv = 1.0f / sqrtf(ss / (float)per + p.eps);
#pragma unroll
    for (int k = 0; k < DN_KEEP; k++) {
        const int i = lane + 32 * k;
        if (i < n) {
            const Pack<4> g = ldp<4>(p.gain + c0 + 4 * i);
            Pack<4> h;
#pragma unroll
            for (int e = 0; e < 4; e++) h.v[e] = keep[k].v[e] * inv * g.v[e];
            if (p.h_out) stp(p.h_out + row + 4 * (size_t)i, h);
            if (p.split) { __nv_bfloat16* hi = static_cast<__nv_bfloat16*>(p.split); split_store4(hi, hi + p.split_lo, row + 4 * (size_t)i, h.v); }
        }
    }
}

// four channels per thread, BF16 tables
__global__ void __launch_bounds__(256) embed_bigram4_kernel(float* __restrict__ x0, float* __restrict__ x1, const __nv_bfloat16* __restrict__ E, const __nv_bfloat16* __restrict__ B,
                                                            const int* __restrict__ tokens, const int* __restrict__ prev, int width, long long buckets, long long mul_prev,
                                                            long long mul_cur, const int* __restrict__ pos_dev, int p0) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.y, i = (blockIdx.x * 256 + threadIdx.x) * 4;
    if (i >= width) return;
    const long long tok = tokens[t];
    auto load = [&](const __nv_bfloat16* p, float (&f)[4]) {
        const uint2 w = *reinterpret_cast<const uint2*>(p);
        f[0] = __uint_as_float(w.x << 16); f[1] = __uint_as_float(w.x & 0xFFFF0000u); f[2] = __uint_as_float(w.y << 16); f[3] = __uint_as_float(w.y & 0xFFFF0000u);
    };
    float a[4], b[4] = {0.f, 0.f, 0.f, 0.f};
    load(E + (size_t)tok * width + i, a);
    if (B) {
        const bool first = t == 0 && (pos_dev ? *pos_dev : p0) == 0;
        long long row = buckets;
        if (!first) {
            const long long before = t > 0 ? tokens[t - 1] : *prev;
            row = (before * mul_prev + tok * mul_cur) % buckets;
            if (row < 0) row += buckets;
        }
        load(B + (size_t)row * width + i, b);
    }
    const float4 v = make_float4(a[0] + b[0], a[1] + b[1], a[2] + b[2], a[3] + b[3]);
    *reinterpret_cast<float4*>(x0 + (size_t)t * width + i) = v;
    if (x1) *reinterpret_cast<float4*>(x1 + (size_t)t * width + i) = v;
}

}  // namespace

void embed_bigram_rows(float* x0, float* x1, const void* E, DType edt, const void* B, DType bdt, const int* tokens_dev, const int* prev_dev, int T, int width,
                       long long buckets, long long mul_prev, long long mul_cur, const int* pos_dev, int p0, cudaStream_t s) {
    if (T <= 0) return;
    NT_CHECK(dense_dtype(edt) && (!B || dense_dtype(bdt)), "embed_bigram_rows: dense tables only");
    NT_CHECK(!B || buckets > 0, "embed_bigram_rows: at least one bucket");
    const uintptr_t bits = reinterpret_cast<uintptr_t>(x0) | reinterpret_cast<uintptr_t>(x1) | reinterpret_cast<uintptr_t>(E) | reinterpret_cast<uintptr_t>(B);
    if (edt == DType::BF16 && (!B || bdt == DType::BF16) && width % 4 == 0 && (bits & 15) == 0) {
        launch_k(embed_bigram4_kernel, dim3((width + 1023) / 1024, T), dim3(256), 0, s, x0, x1, static_cast<const __nv_bfloat16*>(E), static_cast<const __nv_bfloat16*>(B), tokens_dev,
                 prev_dev, width, buckets, mul_prev, mul_cur, pos_dev, p0);
        count_launch();
        return;
    }
    launch_k(embed_bigram_kernel, dim3((width + 255) / 256, T), dim3(256), 0, s, x0, x1, E, (int)edt, B, (int)bdt, tokens_dev, prev_dev, width, buckets, mul_prev, mul_cur,
             pos_dev, p0);
    count_launch();
}

void depth_norm_rows(const DepthNorm& p, int T, cudaStream_t s) {
    if (T <= 0) return;
    NT_CHECK(p.n >= 1 && p.groups >= 1 && p.width % p.groups == 0, "depth_norm_rows: the groups must be equal parts of the row");
    NT_CHECK(p.n_mix == 0 || (T == 1 && p.carried && p.gain && p.n_mix <= DepthNorm::MAX_MIX), "depth_norm_rows: shift blends ride along with one row only");
    const int per = p.width / p.groups;
    bool vec = per % 4 == 0 && p.slot % 4 == 0;
    auto al = [&](const void* q) { if (reinterpret_cast<uintptr_t>(q) & 15) vec = false; };
    al(p.X); al(p.x_out); al(p.h_out); al(p.gain); al(p.split); al(p.carried);
    for (int i = 0; i < p.n_mix; i++) { al(p.mu[i]); al(p.mix_out[i]); }
    const int packs = vec ? per / 4 : per;
    if (vec && T > 1 && packs <= 32 * DN_KEEP) {
        launch_k(depth_norm_warp_kernel, dim3((unsigned)(((size_t)T * p.groups + 7) / 8)), dim3(256), 0, s, p, T * p.groups);
        count_launch();
        return;
    }
    const int threads = std::min(256, (packs + 31) / 32 * 32);
    if (vec) launch_k(depth_norm_kernel<4>, dim3(T, p.groups), dim3(threads), 0, s, p);
    else launch_k(depth_norm_kernel<1>, dim3(T, p.groups), dim3(threads), 0, s, p);
    count_launch();
}

}}  // namespace nt::b200
