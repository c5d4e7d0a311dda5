// postnorm.cu — row-wise pieces of the post-norm block form (engine/layer_spec.h BlockForm::POST_NORM) and of its per-layer token
// input, all F32:
//   add_rmsnorm_rows   x[t] += rms(y[t] + bias) * gain        (a sublayer's output is normed, then joins the residual)
//   glu_bias_mul       out = act(gate + b_g) * (up + b_u)      (biases may be null)
//   side_gate_rows     g[t, j] <- gelu_tanh(g[t, j]) * E[token_t, col0 + j]     (E: a second embedding table, any dense dtype)
//   sandwich_norm_rows x[t] += rms(y[t]) * gain_y; h = rms(x[t]) * gain_h as F32 rows and / or the BF16 split of a GEMM's input: what lies between two
//                      sublayers when a norm sits in front of and behind each; both rows are kept in registers.  sandwich_norm_router: one
//                      decoded token's row, with the router's logits from the same launch
//   sigmoid_gate_rows  o * sigmoid(gate), one gate per run of `per` channels, as F32 rows and / or the split
//   relu2_rows         relu(z)^2, likewise
// One CTA per row; a row is read twice (sum of squares, then the update), both times from L1/L2.
// Compiled WITHOUT --use_fast_math.
#include "kernels_internal.h"
#include "bf16_split.cuh"
#include "ring.cuh"
#include <algorithm>
#include <initializer_list>
#include <cuda_bf16.h>
#include <cuda_fp16.h>

namespace nt { namespace b200 {

namespace {

__device__ __forceinline__ float gelu_tanh_f(float z) { return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }

__global__ void __launch_bounds__(256) add_rmsnorm_rows_kernel(float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ gain,
                                                               const float* __restrict__ bias, int width, float eps) {
    __shared__ float red[8];
    pdl_launch_dependents();
    pdl_wait();
    const size_t t = blockIdx.x;
    const float* yr = y + t * width;
    float ss = 0.f;
    for (int i = threadIdx.x; i < width; i += 256) { const float v = yr[i] + (bias ? bias[i] : 0.f); ss = fmaf(v, v, ss); }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xFFFFFFFFu, ss, o);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int w = 0; w < 8; w++) tot += red[w];
    const float inv = 1.0f / sqrtf(tot / (float)width + eps);
    float* xr = x + t * width;
    for (int i = threadIdx.x; i < width; i += 256) { const float v = yr[i] + (bias ? bias[i] : 0.f); xr[i] += v * inv * gain[i]; }
}

__global__ void glu_bias_mul_kernel(float* __restrict__ out, const float* __restrict__ gate, const float* __restrict__ up, const float* __restrict__ bg,
                                    const float* __restrict__ bu, size_t n, int cols, int gelu) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    const int c = (int)(i % cols);
    const float g = gate[i] + (bg ? bg[c] : 0.f), u = up[i] + (bu ? bu[c] : 0.f);
    out[i] = (gelu ? gelu_tanh_f(g) : silu_f(g)) * u;
}

template <typename ET>
__device__ __forceinline__ float eld(const ET* p, size_t i);
template <> __device__ __forceinline__ float eld<float>(const float* p, size_t i) { return p[i]; }
template <> __device__ __forceinline__ float eld<__half>(const __half* p, size_t i) { return __half2float(p[i]); }
template <> __device__ __forceinline__ float eld<__nv_bfloat16>(const __nv_bfloat16* p, size_t i) { return __bfloat162float(p[i]); }

template <typename ET>
__global__ void side_gate_rows_kernel(float* __restrict__ g, const ET* __restrict__ E, int e_cols, int col0, const int* __restrict__ tokens, size_t n, int dim) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    const size_t t = i / dim, j = i % dim;
    g[i] = gelu_tanh_f(g[i]) * eld<ET>(E, (size_t)tokens[t] * e_cols + col0 + j);
}

// ---- between two sublayers of the sandwich form ----
__device__ __forceinline__ float row_sum(float v, float* red) {        // over the CTA; red [32]
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, o);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float tot = 0.f;
    for (int w = 0; w < (int)(blockDim.x >> 5); w++) tot += red[w];
    return tot;
}
__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float sq4(const float4& v) { return fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w))); }

// KEEP 16-byte pieces of the row per thread.  ROUTER (one row): every CTA works out the whole row, the first one writes it (x_out is not x), and the CTAs
// share the router's rows out: logits[e] = <router row e, h>.
template <int KEEP, bool ROUTER>
__global__ void __launch_bounds__(1024) sandwich_norm_kernel(float* x_out, const float* x, const float* __restrict__ y, const float* __restrict__ gain_y, const float* __restrict__ gain_h,
                                                             float* __restrict__ h, __nv_bfloat16* __restrict__ hi, size_t lo, int width, float eps, const float* __restrict__ router,
                                                             float* __restrict__ logits, int experts) {
    __shared__ float red[32];
    const int n = width / 4, nt = blockDim.x;
    float4 gy[KEEP], gh[KEEP];                     // constants: their way from memory overlaps the producer of y
#pragma unroll
    for (int k = 0; k < KEEP; k++) {
        const int i = threadIdx.x + k * nt;
        gy[k] = (y && i < n) ? ld4(gain_y + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
        gh[k] = (gain_h && i < n) ? ld4(gain_h + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    if (ROUTER) for (int e = blockIdx.x; e < experts; e += gridDim.x) l2_prefetch(router + (size_t)e * width, (size_t)width * sizeof(float), threadIdx.x, nt);
    pdl_launch_dependents();
    pdl_wait();
    const size_t row = ROUTER ? 0 : (size_t)blockIdx.x * width;
    const bool writes = !ROUTER || blockIdx.x == 0;
    float4 xv[KEEP];
#pragma unroll
    for (int k = 0; k < KEEP; k++) { const int i = threadIdx.x + k * nt; xv[k] = i < n ? ld4(x + row + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f); }
    if (y) {
        float4 yv[KEEP];
        float ss = 0.f;
#pragma unroll
        for (int k = 0; k < KEEP; k++) { const int i = threadIdx.x + k * nt; yv[k] = i < n ? ld4(y + row + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f); ss += sq4(yv[k]); }
        const float inv = 1.0f / sqrtf(row_sum(ss, red) / (float)width + eps);
#pragma unroll
        for (int k = 0; k < KEEP; k++) {
            const int i = threadIdx.x + k * nt;
            if (i >= n) continue;
            xv[k].x = fmaf(yv[k].x * inv, gy[k].x, xv[k].x); xv[k].y = fmaf(yv[k].y * inv, gy[k].y, xv[k].y);
            xv[k].z = fmaf(yv[k].z * inv, gy[k].z, xv[k].z); xv[k].w = fmaf(yv[k].w * inv, gy[k].w, xv[k].w);
            if (writes) *reinterpret_cast<float4*>(x_out + row + 4 * i) = xv[k];
        }
    }
    if (!gain_h) return;
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < KEEP; k++) ss += sq4(xv[k]);
    const float inv = 1.0f / sqrtf(row_sum(ss, red) / (float)width + eps);
#pragma unroll
    for (int k = 0; k < KEEP; k++) {
        const int i = threadIdx.x + k * nt;
        if (i >= n) continue;
        const float v[4] = {xv[k].x * inv * gh[k].x, xv[k].y * inv * gh[k].y, xv[k].z * inv * gh[k].z, xv[k].w * inv * gh[k].w};
        if (h && writes) *reinterpret_cast<float4*>(h + row + 4 * i) = make_float4(v[0], v[1], v[2], v[3]);
        if (hi) split_store4(hi, hi + lo, row + 4 * (size_t)i, v);
        if (ROUTER) xv[k] = make_float4(v[0], v[1], v[2], v[3]);
    }
    if (ROUTER) for (int e = blockIdx.x; e < experts; e += gridDim.x) {
        float d = 0.f;
#pragma unroll
        for (int k = 0; k < KEEP; k++) {
            const int i = threadIdx.x + k * nt;
            if (i >= n) continue;
            const float4 r = ld4(router + (size_t)e * width + 4 * i);
            d = fmaf(r.x, xv[k].x, d); d = fmaf(r.y, xv[k].y, d); d = fmaf(r.z, xv[k].z, d); d = fmaf(r.w, xv[k].w, d);
        }
        d = row_sum(d, red);
        if (threadIdx.x == 0) logits[e] = d;
    }
}
// any width and alignment
__global__ void __launch_bounds__(256) sandwich_norm_any_kernel(float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ gain_y, const float* __restrict__ gain_h,
                                                                float* __restrict__ h, __nv_bfloat16* __restrict__ hi, size_t lo, int width, float eps) {
    __shared__ float red[32];
    pdl_launch_dependents();
    pdl_wait();
    const size_t row = (size_t)blockIdx.x * width;
    float inv_y = 0.f, ss = 0.f;
    if (y) {
        for (int i = threadIdx.x; i < width; i += 256) ss = fmaf(y[row + i], y[row + i], ss);
        inv_y = 1.0f / sqrtf(row_sum(ss, red) / (float)width + eps);
    }
    ss = 0.f;
    for (int i = threadIdx.x; i < width; i += 256) {
        float v = x[row + i];
        if (y) { v = fmaf(y[row + i] * inv_y, gain_y[i], v); x[row + i] = v; }
        ss = fmaf(v, v, ss);
    }
    if (!gain_h) return;
    const float inv = 1.0f / sqrtf(row_sum(ss, red) / (float)width + eps);
    for (int i = threadIdx.x; i < width; i += 256) {      // a thread reads back what it wrote itself
        const float v = x[row + i] * inv * gain_h[i];
        if (h) h[row + i] = v;
        if (hi) split_store1(hi, hi + lo, row + i, v);
    }
}

__device__ __forceinline__ float gated(float o, float g) { return o / (1.0f + expf(-g)); }
// four channels per thread; PER: 0 one gate per channel (16-byte loads), 1 one per run of `per` channels
template <int PER>
__global__ void __launch_bounds__(256) sigmoid_gate4_kernel(float* __restrict__ out, __nv_bfloat16* __restrict__ hi, size_t lo, const float* __restrict__ o,
                                                            const float* __restrict__ gate, int ld, int per, size_t n4, int cols4) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t i = (size_t)blockIdx.x * 256 + threadIdx.x;
    if (i >= n4) return;
    const size_t t = i / cols4;
    const int c = (int)(i - t * cols4) * 4;
    const float4 a = ld4(o + 4 * i);
    float g[4];
    if (PER == 0) { const float4 q = ld4(gate + t * ld + c); g[0] = q.x; g[1] = q.y; g[2] = q.z; g[3] = q.w; }
    else {
#pragma unroll
        for (int e = 0; e < 4; e++) g[e] = gate[t * ld + (c + e) / per];
    }
    const float v[4] = {gated(a.x, g[0]), gated(a.y, g[1]), gated(a.z, g[2]), gated(a.w, g[3])};
    if (out) *reinterpret_cast<float4*>(out + 4 * i) = make_float4(v[0], v[1], v[2], v[3]);
    if (hi) split_store4(hi, hi + lo, 4 * i, v);
}
__global__ void __launch_bounds__(256) sigmoid_gate_kernel(float* __restrict__ out, __nv_bfloat16* __restrict__ hi, size_t lo, const float* __restrict__ o,
                                                           const float* __restrict__ gate, int ld, int per, size_t n, int cols) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t i = (size_t)blockIdx.x * 256 + threadIdx.x;
    if (i >= n) return;
    const size_t t = i / cols, c = i % cols;
    const float v = gated(o[i], gate[t * ld + c / per]);
    if (out) out[i] = v;
    if (hi) split_store1(hi, hi + lo, i, v);
}
__global__ void __launch_bounds__(256) relu2_rows_kernel(float* __restrict__ out, __nv_bfloat16* __restrict__ hi, size_t lo, const float* __restrict__ in, size_t n) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t i = (size_t)blockIdx.x * 256 + threadIdx.x;
    if (i >= n) return;
    float v = fmaxf(in[i], 0.f);
    v *= v;
    if (out) out[i] = v;
    if (hi) split_store1(hi, hi + lo, i, v);
}

}  // namespace

void add_rmsnorm_rows(float* x, const float* y, const float* gain, const float* bias, int rows, int width, float eps, cudaStream_t s) {
    if (rows <= 0) return;
    launch_k(add_rmsnorm_rows_kernel, dim3(rows), dim3(256), 0, s, x, y, gain, bias, width, eps);
    count_launch();
}

void glu_bias_mul(float* out, const float* gate, const float* up, const float* gate_bias, const float* up_bias, int rows, int cols, bool gelu, cudaStream_t s) {
    const size_t n = (size_t)rows * cols;
    if (!n) return;
    launch_k(glu_bias_mul_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, s, out, gate, up, gate_bias, up_bias, n, cols, gelu ? 1 : 0);
    count_launch();
}

void side_gate_rows(float* g, const void* E, DType dt, int e_cols, int col0, const int* tokens_dev, int rows, int dim, cudaStream_t s) {
    const size_t n = (size_t)rows * dim;
    if (!n) return;
    const dim3 grid((unsigned)((n + 255) / 256));
    if (dt == DType::F32) launch_k(side_gate_rows_kernel<float>, grid, dim3(256), 0, s, g, static_cast<const float*>(E), e_cols, col0, tokens_dev, n, dim);
    else if (dt == DType::F16) launch_k(side_gate_rows_kernel<__half>, grid, dim3(256), 0, s, g, static_cast<const __half*>(E), e_cols, col0, tokens_dev, n, dim);
    else if (dt == DType::BF16) launch_k(side_gate_rows_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, g, static_cast<const __nv_bfloat16*>(E), e_cols, col0, tokens_dev, n, dim);
    else NT_CHECK(false, "side_gate_rows: dense dtypes only");
    count_launch();
}

void sandwich_norm_rows(float* x, const float* y, const float* gain_y, const float* gain_h, float* h, void* split, int rows, int width, float eps, cudaStream_t s) {
    if (rows <= 0) return;
    NT_CHECK((!y || gain_y) && (!gain_h || h || split), "sandwich_norm_rows: a gain or an output is missing");
    __nv_bfloat16* hi = static_cast<__nv_bfloat16*>(split);
    const size_t lo = split_lo_offset(rows, width);
    uintptr_t bits = 0;
    for (const void* p : {(const void*)x, (const void*)y, (const void*)gain_y, (const void*)gain_h, (const void*)h, (const void*)split}) bits |= reinterpret_cast<uintptr_t>(p);
    const int n = width / 4, most = rows == 1 ? 1024 : 256;        // one row: the whole row in flight at once
    const int threads = std::min(most, (n + 31) / 32 * 32), keep = (n + std::max(threads, 1) - 1) / std::max(threads, 1);
    if (width % 4 == 0 && (bits & 15) == 0 && keep <= 4) {
#define NT_SN(K) launch_k(sandwich_norm_kernel<K, false>, dim3(rows), dim3(threads), 0, s, x, (const float*)x, y, gain_y, gain_h, h, hi, lo, width, eps, (const float*)nullptr, (float*)nullptr, 0)
        if (keep <= 1) NT_SN(1); else if (keep <= 2) NT_SN(2); else NT_SN(4);
#undef NT_SN
    } else launch_k(sandwich_norm_any_kernel, dim3(rows), dim3(256), 0, s, x, y, gain_y, gain_h, h, hi, lo, width, eps);
    count_launch();
}

bool sandwich_norm_router(float* x_out, const float* x, const float* y, const float* gain_y, const float* gain_h, float* h, const float* router, float* logits, int experts, int width,
                          float eps, cudaStream_t s) {
    uintptr_t bits = 0;
    for (const void* p : {(const void*)x_out, (const void*)x, (const void*)y, (const void*)gain_y, (const void*)gain_h, (const void*)h, (const void*)router}) bits |= reinterpret_cast<uintptr_t>(p);
    const int n = width / 4, threads = std::min(1024, (n + 31) / 32 * 32), keep = (n + std::max(threads, 1) - 1) / std::max(threads, 1);
    if (width % 4 != 0 || (bits & 15) != 0 || keep > 4 || keep < 1) return false;
    NT_CHECK(x_out != x && y && gain_y && gain_h && h && experts >= 1, "sandwich_norm_router: a row of its own for the new residual, both norms and the router's rows");
    const int grid = std::min(experts, 64);
#define NT_SR(K) launch_k(sandwich_norm_kernel<K, true>, dim3(grid), dim3(threads), 0, s, x_out, x, y, gain_y, gain_h, h, (__nv_bfloat16*)nullptr, (size_t)0, width, eps, router, logits, experts)
    if (keep <= 1) NT_SR(1); else if (keep <= 2) NT_SR(2); else NT_SR(4);
#undef NT_SR
    count_launch();
    return true;
}

void sigmoid_gate_rows(float* out, void* split, const float* o, const float* gate, int ld, int per, int T, int cols, cudaStream_t s) {
    const size_t n = (size_t)T * cols;
    if (!n) return;
    NT_CHECK(per >= 1 && cols % per == 0, "sigmoid_gate_rows: a gate covers an equal run of channels");
    __nv_bfloat16* hi = static_cast<__nv_bfloat16*>(split);
    const size_t lo = split_lo_offset(T, cols);
    uintptr_t bits = 0;
    for (const void* p : {(const void*)out, (const void*)split, (const void*)o}) bits |= reinterpret_cast<uintptr_t>(p);
    const dim3 grid4((unsigned)((n / 4 + 255) / 256));
    if (cols % 4 == 0 && (bits & 15) == 0 && per == 1 && ld % 4 == 0 && (reinterpret_cast<uintptr_t>(gate) & 15) == 0)
        launch_k(sigmoid_gate4_kernel<0>, grid4, dim3(256), 0, s, out, hi, lo, o, gate, ld, per, n / 4, cols / 4);
    else if (cols % 4 == 0 && (bits & 15) == 0) launch_k(sigmoid_gate4_kernel<1>, grid4, dim3(256), 0, s, out, hi, lo, o, gate, ld, per, n / 4, cols / 4);
    else launch_k(sigmoid_gate_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, s, out, hi, lo, o, gate, ld, per, n, cols);
    count_launch();
}

void relu2_rows(float* out, void* split, const float* in, int T, int cols, cudaStream_t s) {
    const size_t n = (size_t)T * cols;
    if (!n) return;
    launch_k(relu2_rows_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, s, out, static_cast<__nv_bfloat16*>(split), split_lo_offset(T, cols), in, n);
    count_launch();
}

}}  // namespace nt::b200
