// wkv.cu — the WKV time mixer around its projections (engine/layer_spec.h WkvSpec).  Per head with a matrix state S [D, D] in F32
// (key channel d, value channel j), reading the rows r_t, k_t, v_t and the per-channel decay w_t in (0, 1):
//       o_t[j] = sum_d r_t[d] S[d, j] + (sum_d r_t[d] u[d] k_t[d]) v_t[j];      S[d, j] <- w_t[d] S[d, j] + k_t[d] v_t[j]
//   shift_mix_rows   the mixer's inputs m_s[t] = h[t] + (h[t-1] - h[t]) mu_s for several s from one read of h, as F32 rows or as the BF16
//                    split a tensor-core GEMM reads; h[-1] is the carried row (zeros when the step starts at position 0), which then
//                    becomes the step's last row
//   tanh_rows        in place
//   wkv_prep         a <- exp(-exp(a + w0)) in place [T, H * D];  ruk [T, H] = sum_d r u k
//   wkv_rows         the recurrence over the rows of a step.  Every column j of S evolves on its own; LN lanes share a column (dim / LN
//                    state numbers each, in registers).  The carried chain of a row is one multiply-add; the dot products of a tile of
//                    16 rows stay in registers and are reduced together (a halving exchange between the lanes: 15 shuffles for 16 rows
//                    instead of 64).  Rows are staged in tiles of 16 by cp.async into two buffers.  Long steps are cut into segments that run
//                    side by side (two launches: the segments' states, then the rows).
//   wkv_out_norm     o / rms(head) * norm * silu(gate), as F32 rows or as the split of the output projection's input
//   wkv_token        one decoded token in one launch: decay (second low-rank matrix, exponentials), recurrence, head norm and gate; a CTA
//                    per head
// The state [H, D (value), D (key)] is read at the start (zeros when the step starts at position 0) and written back at the end, so a
// prompt cut anywhere continues exactly.  A step's base position is *pos_dev when given (the captured decode step), else p0.
// Everything is F32; compiled WITHOUT --use_fast_math (expf / tanhf / division at full precision).
#include "kernels_internal.h"
#include "bf16_split.cuh"
#include "ring.cuh"
#include "scan_rows.cuh"
#include <cuda_fp16.h>
#include <algorithm>
#include <initializer_list>

namespace nt { namespace b200 {

namespace {

__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float decay_of(float z) { return expf(-expf(z)); }

// ---- shift blends ----
template <bool VEC>
__global__ void __launch_bounds__(256) shift_mix_kernel(ShiftMix p, const float* __restrict__ h, const float* __restrict__ carried, int width, const int* __restrict__ pos_dev, int p0) {
    pdl_launch_dependents();
    pdl_wait();
    constexpr int V = VEC ? 4 : 1;
    const int i = (blockIdx.x * 256 + threadIdx.x) * V, t = blockIdx.y;
    if (i >= width) return;
    const size_t at = (size_t)t * width + i;
    float c[V], d[V];
    if constexpr (VEC) { const float4 f = *reinterpret_cast<const float4*>(h + at); c[0] = f.x; c[1] = f.y; c[2] = f.z; c[3] = f.w; } else c[0] = h[at];
    const bool none = t == 0 && (pos_dev ? *pos_dev : p0) == 0;
    const float* pr = t > 0 ? h + at - width : carried + i;
#pragma unroll
    for (int e = 0; e < V; e++) d[e] = (none ? 0.f : pr[e]) - c[e];
    for (int s = 0; s < p.n; s++) {
        float m[V];
#pragma unroll
        for (int e = 0; e < V; e++) m[e] = fmaf(d[e], p.mu[s][i + e], c[e]);
        if (p.out[s]) {
            if constexpr (VEC) *reinterpret_cast<float4*>(p.out[s] + at) = make_float4(m[0], m[1], m[2], m[3]);
            else p.out[s][at] = m[0];
        }
        if (p.split[s]) {
            __nv_bfloat16* hi = static_cast<__nv_bfloat16*>(p.split[s]);
            if constexpr (VEC) split_store4(hi, hi + p.split_lo, at, m);
            else split_store1(hi, hi + p.split_lo, at, m[0]);
        }
    }
}

__global__ void tanh_kernel(float* __restrict__ x, size_t n) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) x[i] = tanhf(x[i]);
}

// grid (T), 256 threads: a warp per head for the bonus term, all threads for the decays
__global__ void __launch_bounds__(256) wkv_prep_kernel(float* __restrict__ a, float* __restrict__ ruk, const float* __restrict__ r, const float* __restrict__ k,
                                                       const float* __restrict__ w0, const float* __restrict__ u, int heads, int dim) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t t = blockIdx.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n = heads * dim;
    for (int h = warp; h < heads; h += 8) {
        float s = 0.f;
        for (int d = lane; d < dim; d += 32) { const int i = h * dim + d; s = fmaf(r[t * n + i] * u[i], k[t * n + i], s); }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xFFFFFFFFu, s, o);
        if (lane == 0) ruk[t * heads + h] = s;
    }
    for (int i = threadIdx.x; i < n; i += 256) a[t * n + i] = decay_of(a[t * n + i] + w0[i]);
}

// The same for heads of whole 16-byte pieces: LN lanes per (row, head), NV pieces each.
__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <int LN, int NV>
__global__ void __launch_bounds__(256) wkv_prep4_kernel(float* __restrict__ a, float* __restrict__ ruk, const float* __restrict__ r, const float* __restrict__ k,
                                                        const float* __restrict__ w0, const float* __restrict__ u, int rows, int heads, int dim) {
    pdl_launch_dependents();
    pdl_wait();
    const int th = (int)(((size_t)blockIdx.x * 256 + threadIdx.x) / LN), l = threadIdx.x % LN;
    const bool live = th < rows * heads;
    const int h = live ? th % heads : 0;
    const size_t base = (size_t)(live ? th : 0) * dim;
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NV; i++) {
        const int d = 4 * (l + LN * i);
        if (live && d < dim) {
            const float4 R = ld4(r + base + d), K = ld4(k + base + d), U = ld4(u + h * dim + d), O = ld4(w0 + h * dim + d);
            float4 A = ld4(a + base + d);
            s = fmaf(R.x * U.x, K.x, s); s = fmaf(R.y * U.y, K.y, s); s = fmaf(R.z * U.z, K.z, s); s = fmaf(R.w * U.w, K.w, s);
            A.x = decay_of(A.x + O.x); A.y = decay_of(A.y + O.y); A.z = decay_of(A.z + O.z); A.w = decay_of(A.w + O.w);
            *reinterpret_cast<float4*>(a + base + d) = A;
        }
    }
#pragma unroll
    for (int o = LN / 2; o > 0; o >>= 1) s += __shfl_xor_sync(0xFFFFFFFFu, s, o);
    if (l == 0 && live) ruk[th] = s;
}

// ---- recurrence over rows ----
constexpr int WR_TILE = SCAN_TILE;

// grid (ceil(dim / COLS), heads, segments), 128 threads.  LN lanes share CB neighbouring columns: one read of r, k, w from shared memory (what
// bounds the kernel) serves CB columns.  Lane l holds state elements W * (c LN + l) + j, c < CH, j < W, of each.
// PASS 0: the whole step, one segment.  A long step with few columns is cut into segments of seg_len rows that run side by side: the recurrence is
// linear, so the state behind a segment is (product of its decays) * (state in front) + (state from zero).
// PASS 1: segments 0 .. segments - 2, state only: seg[z] <- the state from zero (segment 0: from the real one), decay[z] <- the product of the
//         decays; segment 0 also keeps the step's first state in seg[last].
// PASS 2: every segment joins the states in front of it, then produces its rows; the last one writes the state back.
template <int LN, int CH, int W, int CB, int PASS>
__global__ void __launch_bounds__(128) wkv_rows_kernel(float* __restrict__ out, const float* __restrict__ r, const float* __restrict__ k, const float* __restrict__ v,
                                                       const float* __restrict__ w, const float* __restrict__ ruk, float* __restrict__ state, int T, int heads, int dim,
                                                       const int* __restrict__ pos_dev, int p0, float* __restrict__ seg, float* __restrict__ decay, int seg_len, int segments) {
    constexpr int THREADS = 128, COLS = THREADS / LN * CB, ROWS_LEFT = LN >= WR_TILE ? 1 : WR_TILE / LN;
    extern __shared__ __align__(16) float sm[];
    const int tile_floats = 3 * WR_TILE * dim + WR_TILE * COLS + WR_TILE;      // r | k | w [WR_TILE][dim], v [WR_TILE][COLS], ruk [WR_TILE]
    const int buf_floats = (tile_floats + 3) & ~3;
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.y, n = heads * dim;
    const int col_l = threadIdx.x / LN * CB, l = threadIdx.x % LN;
    const int col = blockIdx.x * COLS + col_l;
    const bool fresh = (pos_dev ? *pos_dev : p0) == 0;
    const size_t all = (size_t)heads * dim * dim;
    auto st_off = [&](int b) { return ((size_t)h * dim + col + b) * dim; };       // only for live columns, col + b < dim
    const int z = PASS == 0 ? 0 : blockIdx.z;
    if (PASS != 0) {                            // this segment's rows
        const size_t first = (size_t)z * seg_len;
        r += first * n; k += first * n; v += first * n; w += first * n; ruk += first * heads; out += first * n;
        T = min(seg_len, T - z * seg_len);
    }
    int d0[CH];
    bool on[CH];
    float S[CB][CH][W], prod[PASS == 1 ? CH : 1][W];
#pragma unroll
    for (int c = 0; c < CH; c++) {
        d0[c] = W * (c * LN + l);
        on[c] = d0[c] < dim;
        if (PASS == 1) {
#pragma unroll
            for (int j = 0; j < W; j++) prod[c][j] = 1.f;
        }
#pragma unroll
        for (int b = 0; b < CB; b++) {
#pragma unroll
            for (int j = 0; j < W; j++) S[b][c][j] = 0.f;
            if (!on[c] || col + b >= dim) continue;
            const size_t at = st_off(b) + d0[c];
            if (PASS != 2 && z == 0) {
#pragma unroll
                for (int j = 0; j < W; j++) {
                    if (!fresh) S[b][c][j] = state[at + j];
                    if (PASS == 1) seg[(size_t)(segments - 1) * all + at + j] = S[b][c][j];
                }
            }
            if (PASS == 2) {
                const float* from = seg + (z == 0 ? (size_t)(segments - 1) * all : 0) + at;
#pragma unroll
                for (int j = 0; j < W; j++) S[b][c][j] = from[j];
                for (int y = 1; y < z; y++) {
#pragma unroll
                    for (int j = 0; j < W; j++) S[b][c][j] = fmaf(decay[((size_t)y * heads + h) * dim + d0[c] + j], S[b][c][j], seg[(size_t)y * all + at + j]);
                }
            }
        }
        if (!on[c]) d0[c] = 0;
    }
    auto load_tile = [&](int t0, int buf) {
        float* sr = sm + (size_t)buf * buf_floats;
        float* sk = sr + WR_TILE * dim;
        float* sw = sk + WR_TILE * dim;
        float* sv = sw + WR_TILE * dim;
        float* sb = sv + WR_TILE * COLS;
        const int nt = min(WR_TILE, T - t0), dv = dim / W;
        for (int i = threadIdx.x; i < nt * dv; i += THREADS) {
            const int tt = i / dv, d = (i - tt * dv) * W;
            const size_t at = (size_t)(t0 + tt) * n + (size_t)h * dim + d;
            if constexpr (W == 4) { if (PASS != 1) cp_async16(sr + tt * dim + d, r + at); cp_async16(sk + tt * dim + d, k + at); cp_async16(sw + tt * dim + d, w + at); }
            else { if (PASS != 1) cp_async4(sr + tt * dim + d, r + at); cp_async4(sk + tt * dim + d, k + at); cp_async4(sw + tt * dim + d, w + at); }
        }
        for (int i = threadIdx.x; i < nt * COLS; i += THREADS) {
            const int tt = i / COLS, c = blockIdx.x * COLS + i % COLS;
            if (c < dim) cp_async4(sv + i, v + (size_t)(t0 + tt) * n + (size_t)h * dim + c);
            else sv[i] = 0.f;
        }
        if (PASS != 1) for (int i = threadIdx.x; i < nt; i += THREADS) cp_async4(sb + i, ruk + (size_t)(t0 + i) * heads + h);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    const int n_tiles = (T + WR_TILE - 1) / WR_TILE;
    load_tile(0, 0);
    for (int q = 0; q < n_tiles; q++) {
        const int t0 = q * WR_TILE, nt = min(WR_TILE, T - t0), buf = q & 1;
        if (q + 1 < n_tiles) {
            load_tile(t0 + WR_TILE, buf ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const float* sr = sm + (size_t)buf * buf_floats;
        const float* sk = sr + WR_TILE * dim;
        const float* sw = sk + WR_TILE * dim;
        const float* sv = sw + WR_TILE * dim;
        const float* sb = sv + WR_TILE * COLS;
        float part[CB][WR_TILE];
        auto step = [&](int tt) {
            float vj[CB], p[CB];
#pragma unroll
            for (int b = 0; b < CB; b++) { vj[b] = sv[tt * COLS + col_l + b]; p[b] = 0.f; }
#pragma unroll
            for (int c = 0; c < CH; c++) {
                float rr[W], kk[W], ww[W];
                if constexpr (W == 4) {
                    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
                    if (PASS != 1) a = *reinterpret_cast<const float4*>(sr + tt * dim + d0[c]);
                    const float4 b = *reinterpret_cast<const float4*>(sk + tt * dim + d0[c]), e = *reinterpret_cast<const float4*>(sw + tt * dim + d0[c]);
                    rr[0] = a.x; rr[1] = a.y; rr[2] = a.z; rr[3] = a.w; kk[0] = b.x; kk[1] = b.y; kk[2] = b.z; kk[3] = b.w; ww[0] = e.x; ww[1] = e.y; ww[2] = e.z; ww[3] = e.w;
                } else { rr[0] = PASS != 1 ? sr[tt * dim + d0[c]] : 0.f; kk[0] = sk[tt * dim + d0[c]]; ww[0] = sw[tt * dim + d0[c]]; }
                if (CH == 1 || on[c]) {
#pragma unroll
                    for (int j = 0; j < W; j++) {
#pragma unroll
                        for (int b = 0; b < CB; b++) {
                            if (PASS != 1) p[b] = fmaf(rr[j], S[b][c][j], p[b]);
                            S[b][c][j] = fmaf(ww[j], S[b][c][j], kk[j] * vj[b]);
                        }
                        if (PASS == 1) prod[c][j] *= ww[j];
                    }
                }
            }
#pragma unroll
            for (int b = 0; b < CB; b++) part[b][tt] = (CH == 1 && !on[0]) ? 0.f : p[b];
        };
        if (nt == WR_TILE) {
#pragma unroll
            for (int tt = 0; tt < WR_TILE; tt++) step(tt);
        } else {
#pragma unroll
            for (int tt = 0; tt < WR_TILE; tt++) {
                if (tt < nt) step(tt);
                else {
#pragma unroll
                    for (int b = 0; b < CB; b++) part[b][tt] = 0.f;
                }
            }
        }
        if (PASS != 1) {
#pragma unroll
            for (int b = 0; b < CB; b++) {
                const int row0 = reduce_rows<LN>(part[b], l);
#pragma unroll
                for (int j = 0; j < ROWS_LEFT; j++) {
                    const int tt = row0 + j;
                    if (col + b < dim && tt < nt && (LN <= WR_TILE || (l & 1) == 0))
                        out[(size_t)(t0 + tt) * n + (size_t)h * dim + col + b] = fmaf(sb[tt], sv[tt * COLS + col_l + b], part[b][j]);
                }
            }
        }
        __syncthreads();                       // the buffer is refilled by the load of tile q + 2
    }
    if (PASS == 2 && z != segments - 1) return;
    float* to = PASS == 1 ? seg + (size_t)z * all : state;
#pragma unroll
    for (int c = 0; c < CH; c++) {
        if (!on[c]) continue;
#pragma unroll
        for (int b = 0; b < CB; b++) {
            if (col + b >= dim) continue;
#pragma unroll
            for (int j = 0; j < W; j++) to[st_off(b) + d0[c] + j] = S[b][c][j];
        }
        if (PASS == 1 && col == 0) {
#pragma unroll
            for (int j = 0; j < W; j++) decay[((size_t)z * heads + h) * dim + d0[c] + j] = prod[c][j];
        }
    }
}

// grid (T), 256 threads, a warp per head
__global__ void __launch_bounds__(256) wkv_out_norm_kernel(float* __restrict__ out, __nv_bfloat16* __restrict__ hi, size_t lo_off, const float* __restrict__ o,
                                                           const float* __restrict__ gate, const float* __restrict__ norm, float eps, int heads, int dim) {
    pdl_launch_dependents();
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const size_t row = (size_t)blockIdx.x * heads * dim;
    for (int h = warp; h < heads; h += 8) {
        const float* oh = o + row + (size_t)h * dim;
        float ss = 0.f;
        for (int d = lane; d < dim; d += 32) ss = fmaf(oh[d], oh[d], ss);
#pragma unroll
        for (int q = 16; q > 0; q >>= 1) ss += __shfl_xor_sync(0xFFFFFFFFu, ss, q);
        const float inv = 1.0f / sqrtf(ss / (float)dim + eps);
        for (int d = lane; d < dim; d += 32) {
            const int c = h * dim + d;
            const float y = oh[d] * inv * norm[c] * silu_f(gate[row + c]);
            if (out) out[row + c] = y;
            if (hi) split_store1(hi, hi + lo_off, row + c, y);
        }
    }
}

// The same for heads of whole 16-byte pieces: LN lanes per (row, head), NV pieces each.
template <int LN, int NV>
__global__ void __launch_bounds__(256) wkv_out_norm4_kernel(float* __restrict__ out, __nv_bfloat16* __restrict__ hi, size_t lo_off, const float* __restrict__ o,
                                                            const float* __restrict__ gate, const float* __restrict__ norm, float eps, int rows, int heads, int dim) {
    pdl_launch_dependents();
    pdl_wait();
    const int th = (int)(((size_t)blockIdx.x * 256 + threadIdx.x) / LN), l = threadIdx.x % LN;
    const bool live = th < rows * heads;
    const int h = live ? th % heads : 0;
    const size_t base = (size_t)(live ? th : 0) * dim;
    float4 v[NV];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; i++) {
        const int d = 4 * (l + LN * i);
        v[i] = (live && d < dim) ? ld4(o + base + d) : make_float4(0.f, 0.f, 0.f, 0.f);
        ss = fmaf(v[i].x, v[i].x, ss); ss = fmaf(v[i].y, v[i].y, ss); ss = fmaf(v[i].z, v[i].z, ss); ss = fmaf(v[i].w, v[i].w, ss);
    }
#pragma unroll
    for (int q = LN / 2; q > 0; q >>= 1) ss += __shfl_xor_sync(0xFFFFFFFFu, ss, q);
    const float inv = 1.0f / sqrtf(ss / (float)dim + eps);
#pragma unroll
    for (int i = 0; i < NV; i++) {
        const int d = 4 * (l + LN * i);
        if (live && d < dim) {
            const float4 N = ld4(norm + h * dim + d), G = ld4(gate + base + d);
            const float y[4] = {v[i].x * inv * N.x * silu_f(G.x), v[i].y * inv * N.y * silu_f(G.y), v[i].z * inv * N.z * silu_f(G.z), v[i].w * inv * N.w * silu_f(G.w)};
            if (out) *reinterpret_cast<float4*>(out + base + d) = make_float4(y[0], y[1], y[2], y[3]);
            if (hi) split_store4(hi, hi + lo_off, base + d, y);
        }
    }
}

__device__ __forceinline__ float wld(const float* p, size_t i) { return __ldg(p + i); }
__device__ __forceinline__ float wld(const __half* p, size_t i) { return __half2float(__ushort_as_half(__ldg(reinterpret_cast<const unsigned short*>(p) + i))); }
__device__ __forceinline__ float wld(const __nv_bfloat16* p, size_t i) { return __uint_as_float((unsigned)__ldg(reinterpret_cast<const unsigned short*>(p) + i) << 16); }

template <typename T> struct Chunk;           // 16 bytes of a weight row
template <> struct Chunk<float> {
    static constexpr int P = 4;
    static __device__ __forceinline__ void unpack(const uint4& w, float* f) { f[0] = __uint_as_float(w.x); f[1] = __uint_as_float(w.y); f[2] = __uint_as_float(w.z); f[3] = __uint_as_float(w.w); }
};
template <> struct Chunk<__half> {
    static constexpr int P = 8;
    static __device__ __forceinline__ void unpack(const uint4& w, float* f) {
        const unsigned u[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
        for (int k = 0; k < 4; k++) { const float2 p = __half22float2(*reinterpret_cast<const __half2*>(&u[k])); f[2 * k] = p.x; f[2 * k + 1] = p.y; }
    }
};
template <> struct Chunk<__nv_bfloat16> {
    static constexpr int P = 8;
    static __device__ __forceinline__ void unpack(const uint4& w, float* f) {
        const unsigned u[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
        for (int k = 0; k < 4; k++) { f[2 * k] = __uint_as_float(u[k] << 16); f[2 * k + 1] = __uint_as_float(u[k] & 0xFFFF0000u); }
    }
};

// grid (heads), 256 threads.  a1 [rank]: tanh(W_w1 m) of the token; W2 [heads * dim, rank].  8 lanes per value channel; DV > 0: dim is a
// multiple of 4 and at most 32 DV, a lane's share of a column is DV 16-byte pieces loaded together; DV == 0: any dim.  vec: W2's rows are whole
// 16-byte pieces, 8 lanes per row.
constexpr int WT_LN = 8;
template <typename T, int DV>
__global__ void __launch_bounds__(256) wkv_token_kernel(float* __restrict__ out, const float* __restrict__ r, const float* __restrict__ k, const float* __restrict__ v,
                                                        const float* __restrict__ gate, const float* __restrict__ a1, const T* __restrict__ W2, const float* __restrict__ w0,
                                                        const float* __restrict__ u, const float* __restrict__ norm, float* __restrict__ state, float eps, int rank,
                                                        int dim, int vec, const int* __restrict__ pos_dev, int p0) {
    extern __shared__ __align__(16) float sm[];
    const int dp = (dim + 3) & ~3;
    float *rs = sm, *ks = rs + dp, *ws = ks + dp, *os = ws + dp, *as = os + dp;      // [dim] x 4, [rank]
    __shared__ float red[8];
    __shared__ float bonus;
    const int h = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const size_t hb = (size_t)h * dim;
    // the state and the constants are older than this step: their way from HBM overlaps the projections
    l2_prefetch(state + hb * dim, (size_t)dim * dim * sizeof(float), threadIdx.x, 256);
    l2_prefetch(W2 + hb * rank, (size_t)dim * rank * sizeof(T), threadIdx.x, 256);
    l2_prefetch(w0 + hb, (size_t)dim * sizeof(float), threadIdx.x, 256);
    l2_prefetch(u + hb, (size_t)dim * sizeof(float), threadIdx.x, 256);
    l2_prefetch(norm + hb, (size_t)dim * sizeof(float), threadIdx.x, 256);
    pdl_launch_dependents();
    pdl_wait();
    const bool fresh = (pos_dev ? *pos_dev : p0) == 0;
    for (int i = threadIdx.x; i < rank; i += 256) as[i] = a1[i];
    for (int d = threadIdx.x; d < dim; d += 256) { rs[d] = r[hb + d]; ks[d] = k[hb + d]; }
    __syncthreads();
    const int l = threadIdx.x % WT_LN;
    if (vec) {
        constexpr int P = Chunk<T>::P;
        const int nc = rank / P;
#pragma unroll 2
        for (int d0 = 0; d0 < dim; d0 += 256 / WT_LN) {
            const int d = d0 + threadIdx.x / WT_LN;
            float z = 0.f;
            if (d < dim) {
                const uint4* row = reinterpret_cast<const uint4*>(W2 + (hb + d) * rank);
                for (int c = l; c < nc; c += WT_LN) {
                    float f[P];
                    Chunk<T>::unpack(__ldg(row + c), f);
#pragma unroll
                    for (int e = 0; e < P; e++) z = fmaf(f[e], as[c * P + e], z);
                }
            }
#pragma unroll
            for (int o = WT_LN / 2; o > 0; o >>= 1) z += __shfl_xor_sync(0xFFFFFFFFu, z, o);
            if (l == 0 && d < dim) ws[d] = decay_of(z + w0[hb + d]);
        }
    } else {
        for (int d = warp; d < dim; d += 8) {
            float z = 0.f;
            for (int i = lane; i < rank; i += 32) z = fmaf(wld(W2, (hb + d) * rank + i), as[i], z);
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) z += __shfl_xor_sync(0xFFFFFFFFu, z, o);
            if (lane == 0) ws[d] = decay_of(z + w0[hb + d]);
        }
    }
    if (warp == 0) {
        float s = 0.f;
        for (int d = lane; d < dim; d += 32) s = fmaf(rs[d] * u[hb + d], ks[d], s);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xFFFFFFFFu, s, o);
        if (lane == 0) bonus = s;
    }
    __syncthreads();
#pragma unroll 2
    for (int j0 = 0; j0 < dim; j0 += 256 / WT_LN) {
        const int j = j0 + threadIdx.x / WT_LN;
        const bool live = j < dim;
        float* st = state + (hb + (live ? j : 0)) * dim;
        const float vj = live ? v[hb + j] : 0.f;
        float p = 0.f;
        if constexpr (DV > 0) {
            float4 S[DV];
#pragma unroll
            for (int c = 0; c < DV; c++) {
                const int d = 4 * (c * WT_LN + l);
                S[c] = (live && !fresh && d < dim) ? *reinterpret_cast<const float4*>(st + d) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
#pragma unroll
            for (int c = 0; c < DV; c++) {
                const int d = 4 * (c * WT_LN + l);
                if (live && d < dim) {
                    const float4 R = *reinterpret_cast<const float4*>(rs + d), K = *reinterpret_cast<const float4*>(ks + d), D = *reinterpret_cast<const float4*>(ws + d);
                    p = fmaf(R.x, S[c].x, p); p = fmaf(R.y, S[c].y, p); p = fmaf(R.z, S[c].z, p); p = fmaf(R.w, S[c].w, p);
                    S[c].x = fmaf(D.x, S[c].x, K.x * vj); S[c].y = fmaf(D.y, S[c].y, K.y * vj); S[c].z = fmaf(D.z, S[c].z, K.z * vj); S[c].w = fmaf(D.w, S[c].w, K.w * vj);
                    *reinterpret_cast<float4*>(st + d) = S[c];
                }
            }
        } else {
            for (int d = l; live && d < dim; d += WT_LN) {
                const float S = fresh ? 0.f : st[d];
                p = fmaf(rs[d], S, p);
                st[d] = fmaf(ws[d], S, ks[d] * vj);
            }
        }
#pragma unroll
        for (int o = WT_LN / 2; o > 0; o >>= 1) p += __shfl_xor_sync(0xFFFFFFFFu, p, o);
        if (l == 0 && live) os[j] = fmaf(bonus, vj, p);
    }
    __syncthreads();
    float ss = 0.f;
    for (int d = threadIdx.x; d < dim; d += 256) ss = fmaf(os[d], os[d], ss);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xFFFFFFFFu, ss, o);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int w = 0; w < 8; w++) tot += red[w];
    const float inv = 1.0f / sqrtf(tot / (float)dim + eps);
    for (int d = threadIdx.x; d < dim; d += 256) out[hb + d] = os[d] * inv * norm[hb + d] * silu_f(gate[hb + d]);
}

constexpr int WR_MAX_SEGMENTS = 8;
template <int LN, int CH, int W, int CB>
void launch_rows(float* out, const float* r, const float* k, const float* v, const float* w, const float* ruk, float* state, int T, int heads, int dim, const int* pos_dev,
                 int p0, float* scratch, cudaStream_t s) {
    constexpr int COLS = 128 / LN * CB;
    const size_t tile = ((size_t)3 * WR_TILE * dim + (size_t)WR_TILE * COLS + WR_TILE + 3) & ~(size_t)3;
    const size_t smem = sizeof(float) * 2 * tile;
    const int cols = (dim + COLS - 1) / COLS;
    // segments where the columns leave half of the SMs without a CTA: until about six CTAs stand on every SM, none shorter than eight tiles.  The
    // state pass costs about half of a full one, so a grid that fills the SMs on its own, or two segments, gain nothing.
    int segments = 1;
    if (scratch && 2 * cols * heads <= 148) segments = std::max(1, std::min({WR_MAX_SEGMENTS, (6 * 148 + cols * heads - 1) / (cols * heads), T / (8 * WR_TILE)}));
    if (segments < 3) segments = 1;
    const int seg_len = ((T + segments - 1) / segments + WR_TILE - 1) / WR_TILE * WR_TILE;
    segments = (T + seg_len - 1) / seg_len;
    static unsigned long long done0 = 0, done1 = 0, done2 = 0;
    if (segments == 1) {
        if (smem > 48 * 1024) opt_in_dynamic_smem(wkv_rows_kernel<LN, CH, W, CB, 0>, 200 * 1024, done0);
        launch_k(wkv_rows_kernel<LN, CH, W, CB, 0>, dim3(cols, heads), dim3(128), smem, s, out, r, k, v, w, ruk, state, T, heads, dim, pos_dev, p0, (float*)nullptr, (float*)nullptr, T, 1);
        count_launch();
        return;
    }
    float* decay = scratch + (size_t)WR_MAX_SEGMENTS * heads * dim * dim;
    if (smem > 48 * 1024) { opt_in_dynamic_smem(wkv_rows_kernel<LN, CH, W, CB, 1>, 200 * 1024, done1); opt_in_dynamic_smem(wkv_rows_kernel<LN, CH, W, CB, 2>, 200 * 1024, done2); }
    launch_k(wkv_rows_kernel<LN, CH, W, CB, 1>, dim3(cols, heads, segments - 1), dim3(128), smem, s, out, r, k, v, w, ruk, state, T, heads, dim, pos_dev, p0, scratch, decay, seg_len, segments);
    launch_k(wkv_rows_kernel<LN, CH, W, CB, 2>, dim3(cols, heads, segments), dim3(128), smem, s, out, r, k, v, w, ruk, state, T, heads, dim, pos_dev, p0, scratch, decay, seg_len, segments);
    count_launch(2);
}

}  // namespace

void shift_mix_rows(const ShiftMix& p, const float* h, float* carried, int T, int width, const int* pos_dev, int p0, cudaStream_t s) {
    if (T <= 0) return;
    NT_CHECK(p.n >= 1 && p.n <= ShiftMix::MAX, "shift_mix_rows: 1..5 blends");
    bool vec = width % 4 == 0;
    auto al = [&](const void* q) { if (reinterpret_cast<uintptr_t>(q) & 15) vec = false; };
    al(h); al(carried);
    for (int i = 0; i < p.n; i++) { al(p.mu[i]); al(p.out[i]); al(p.split[i]); }
    const int per = vec ? 1024 : 256;
    const dim3 grid((width + per - 1) / per, T);
    if (vec) launch_k(shift_mix_kernel<true>, grid, dim3(256), 0, s, p, h, (const float*)carried, width, pos_dev, p0);
    else launch_k(shift_mix_kernel<false>, grid, dim3(256), 0, s, p, h, (const float*)carried, width, pos_dev, p0);
    count_launch();
    copy(carried, h + (size_t)(T - 1) * width, width, s);
}

void tanh_rows(float* x, size_t n, cudaStream_t s) {
    if (!n) return;
    launch_k(tanh_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, s, x, n);
    count_launch();
}

void wkv_prep(float* a, float* ruk, const float* r, const float* k, const float* w0, const float* u, int T, int heads, int dim, cudaStream_t s) {
    if (T <= 0) return;
    const auto al = [](std::initializer_list<const void*> ps) { uintptr_t b = 0; for (const void* p : ps) b |= reinterpret_cast<uintptr_t>(p); return (b & 15) == 0; };
    if (dim % 4 == 0 && dim <= 256 && al({a, r, k, w0, u})) {
#define NT_WP(LN, NV) launch_k(wkv_prep4_kernel<LN, NV>, dim3((unsigned)(((size_t)T * heads * LN + 255) / 256)), dim3(256), 0, s, a, ruk, r, k, w0, u, T, heads, dim)
        if (dim <= 16) NT_WP(4, 1); else if (dim <= 32) NT_WP(8, 1); else if (dim <= 64) NT_WP(16, 1); else if (dim <= 128) NT_WP(32, 1); else NT_WP(32, 2);
#undef NT_WP
        count_launch();
        return;
    }
    launch_k(wkv_prep_kernel, dim3(T), dim3(256), 0, s, a, ruk, r, k, w0, u, heads, dim);
    count_launch();
}

size_t wkv_rows_scratch_floats(int heads, int dim) { return (size_t)WR_MAX_SEGMENTS * heads * dim * ((size_t)dim + 1); }

void wkv_rows(float* out, const float* r, const float* k, const float* v, const float* w, const float* ruk, float* state, int T, int heads, int dim, const int* pos_dev, int p0,
              cudaStream_t s, float* scratch) {
    NT_CHECK(dim >= 1 && dim <= WKV_MAX_DIM, "wkv_rows: heads wider than 256 are not covered");
    if (T <= 0) return;
    const bool vec = dim % 4 == 0 && ((reinterpret_cast<uintptr_t>(r) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(w)) & 15) == 0;
#define NT_WR(LN, CH, W, CB) launch_rows<LN, CH, W, CB>(out, r, k, v, w, ruk, state, T, heads, dim, pos_dev, p0, scratch, s)
    if (vec) {
        if (dim <= 16) NT_WR(4, 1, 4, 1);
        else if (dim <= 32) NT_WR(8, 1, 4, 2);
        else if (dim <= 64) NT_WR(16, 1, 4, 4);
        else if (dim <= 128) NT_WR(16, 2, 4, 2);
        else NT_WR(32, 2, 4, 2);
    } else {
        if (dim <= 8) NT_WR(8, 1, 1, 1);
        else if (dim <= 32) NT_WR(16, 2, 1, 1);
        else if (dim <= 128) NT_WR(16, 8, 1, 1);
        else NT_WR(16, 16, 1, 1);
    }
#undef NT_WR
}

void wkv_out_norm(float* out, void* split, const float* o, const float* gate, const float* norm, float eps, int T, int heads, int dim, cudaStream_t s) {
    if (T <= 0) return;
    const auto al = [](std::initializer_list<const void*> ps) { uintptr_t b = 0; for (const void* p : ps) b |= reinterpret_cast<uintptr_t>(p); return (b & 15) == 0; };
    if (dim % 4 == 0 && dim <= 256 && al({out, split, o, gate, norm})) {
#define NT_WN(LN, NV) launch_k(wkv_out_norm4_kernel<LN, NV>, dim3((unsigned)(((size_t)T * heads * LN + 255) / 256)), dim3(256), 0, s, out, static_cast<__nv_bfloat16*>(split), \
                               split_lo_offset(T, heads * dim), o, gate, norm, eps, T, heads, dim)
        if (dim <= 16) NT_WN(4, 1); else if (dim <= 32) NT_WN(8, 1); else if (dim <= 64) NT_WN(16, 1); else if (dim <= 128) NT_WN(32, 1); else NT_WN(32, 2);
#undef NT_WN
        count_launch();
        return;
    }
    launch_k(wkv_out_norm_kernel, dim3(T), dim3(256), 0, s, out, static_cast<__nv_bfloat16*>(split), split_lo_offset(T, heads * dim), o, gate, norm, eps, heads, dim);
    count_launch();
}

void wkv_token(float* out, const float* r, const float* k, const float* v, const float* gate, const float* a1, const void* W2, DType dt, const float* w0, const float* u,
               const float* norm, float* state, float eps, int rank, int heads, int dim, const int* pos_dev, int p0, cudaStream_t s) {
    NT_CHECK(dim >= 1 && dim <= WKV_MAX_DIM && rank >= 1, "wkv_token: heads wider than 256 are not covered");
    const size_t smem = sizeof(float) * (4 * (size_t)((dim + 3) & ~3) + (size_t)rank);
    NT_CHECK(smem <= 48 * 1024, "wkv_token: decay ranks above 11000 are not covered");
    NT_CHECK(dense_dtype(dt), "wkv_token: dense dtypes only");
    const int vec = rank % (dt == DType::F32 ? 4 : 8) == 0 && (reinterpret_cast<uintptr_t>(W2) & 15) == 0;
    const int dv = dim % 4 || (reinterpret_cast<uintptr_t>(state) & 15) ? 0 : dim <= 32 ? 1 : dim <= 64 ? 2 : dim <= 128 ? 4 : 8;
#define NT_WD(TY, DV) launch_k(wkv_token_kernel<TY, DV>, dim3(heads), dim3(256), smem, s, out, r, k, v, gate, a1, static_cast<const TY*>(W2), w0, u, norm, state, eps, rank, dim, vec, pos_dev, p0)
#define NT_WT(TY) { if (dv == 1) NT_WD(TY, 1); else if (dv == 2) NT_WD(TY, 2); else if (dv == 4) NT_WD(TY, 4); else if (dv == 8) NT_WD(TY, 8); else NT_WD(TY, 0); }
    if (dt == DType::F32) NT_WT(float) else if (dt == DType::F16) NT_WT(__half) else NT_WT(__nv_bfloat16)
#undef NT_WD
#undef NT_WT
    count_launch();
}

}}  // namespace nt::b200
