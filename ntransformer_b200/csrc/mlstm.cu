// mlstm.cu — matrix memory with exponential gates around its projections (engine/layer_spec.h MlstmSpec).  Per head with S [D, V] (key channel d, value
// channel j), normalizer n [D] and stabilizer m, log input gate i_t and log forget gate f_t:
//       m_t = max(f_t + m_(t-1), i_t),   a_t = e^(f_t + m_(t-1) - m_t),   b_t = e^(i_t - m_t)
//       S[d, j] <- a_t S[d, j] + k_t[d] b_t v_t[j],   n[d] <- a_t n[d] + b_t k_t[d],   o_t[j] = sum_d q_t[d] S[d, j] / (max(|<n, q_t>|, e^-m_t) + 1e-6)
// n is one more value channel whose value is 1: the state is [H, V + 1, D] with row V the normalizer, and <n, q> falls out like any other column.
//   mlstm_gates      a, b, e^-m for every row of a step: the recurrence of m is a composition of maps m -> max(F + m, M), scanned over the CTA (a
//                    head each).  The results a and b are formed from consecutive m of the same sequence, so they fit together exactly whatever the
//                    order of the scan's sums.
//   mlstm_rows       the recurrence over the rows of a step.  Every column j evolves on its own; LN lanes share CB neighbouring columns (dim / LN
//                    state numbers of each per lane, in registers), one read of q and k from shared memory serves CB columns.  The dot products of a
//                    tile of 16 rows stay in registers and are reduced together (scan_rows.cuh).  Rows are staged in tiles by cp.async into two
//                    buffers.  Long steps are cut into segments that run side by side (two launches: the segments' states, then the rows).
//   mlstm_out_norm   the quotient, the head norm and the output gate, as F32 rows or as the split of the output projection's input
//   mlstm_token      one decoded token in one launch; the value channels of a head are shared out over the CTAs of a cluster, whose sums of squares
//                    meet through distributed shared memory
// The state is read at the start (zeros when the step starts at position 0) and written back at the end, so a prompt cut anywhere continues exactly.
// A step's base position is *pos_dev when given (the captured decode step), else p0.  Everything is F32; compiled WITHOUT --use_fast_math.
#include "kernels_internal.h"
#include "bf16_split.cuh"
#include "ring.cuh"
#include "scan_rows.cuh"
#include <cooperative_groups.h>
#include <algorithm>
#include <initializer_list>

namespace nt { namespace b200 {

namespace {

__device__ __forceinline__ float capped(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
constexpr float kDenEps = 1e-6f;

// ---- gates ----
struct MaxPlus { float F, M; };                                     // m -> max(F + m, M)
__device__ __forceinline__ MaxPlus then(const MaxPlus& a, const MaxPlus& b) { return {a.F + b.F, fmaxf(a.M + b.F, b.M)}; }      // first a, then b

// grid (heads), GT_THREADS threads: the log gates of all rows first (independent loads in flight together), then a thread composes a run of consecutive
// rows and the runs are scanned over the CTA
constexpr int GT_THREADS = 512;
__global__ void __launch_bounds__(GT_THREADS) mlstm_gates_kernel(float* __restrict__ a, float* __restrict__ b, float* __restrict__ em, const float* __restrict__ zi,
                                                          const float* __restrict__ zf, int ld, const float* __restrict__ bi, const float* __restrict__ bf, float cap,
                                                          float* __restrict__ m_state, int T, int heads, const int* __restrict__ pos_dev, int p0) {
    __shared__ MaxPlus warp_tot[GT_THREADS / 32];
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int per = (T + GT_THREADS - 1) / GT_THREADS, t0 = min(T, (int)threadIdx.x * per), t1 = min(T, t0 + per);
    const float m0 = (pos_dev ? *pos_dev : p0) == 0 ? 0.f : m_state[h], bih = bi[h], bfh = bf[h];
    MaxPlus run = {0.f, -INFINITY};                                 // the identity
#pragma unroll 4
    for (int t = threadIdx.x; t < T; t += GT_THREADS) {
        a[(size_t)t * heads + h] = log_sigmoid(capped(zf[(size_t)t * ld + h] + bfh, cap));
        b[(size_t)t * heads + h] = capped(zi[(size_t)t * ld + h] + bih, cap);
    }
    __syncthreads();
    for (int t = t0; t < t1; t++) run = then(run, {a[(size_t)t * heads + h], b[(size_t)t * heads + h]});
    MaxPlus inc = run;                                              // inclusive scan over the warp, then over the warps
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const MaxPlus prev = {__shfl_up_sync(0xFFFFFFFFu, inc.F, o), __shfl_up_sync(0xFFFFFFFFu, inc.M, o)};
        if (lane >= o) inc = then(prev, inc);
    }
    if (lane == 31) warp_tot[warp] = inc;
    MaxPlus before = {__shfl_up_sync(0xFFFFFFFFu, inc.F, 1), __shfl_up_sync(0xFFFFFFFFu, inc.M, 1)};
    if (lane == 0) before = {0.f, -INFINITY};
    __syncthreads();
    MaxPlus ahead = {0.f, -INFINITY};
    for (int w = 0; w < warp; w++) ahead = then(ahead, warp_tot[w]);
    before = then(ahead, before);
    float m = fmaxf(before.F + m0, before.M);
    for (int t = t0; t < t1; t++) {                                 // the run's numbers are this thread's alone by now
        const size_t at = (size_t)t * heads + h;
        const float f = a[at], i = b[at], mn = fmaxf(f + m, i);
        a[at] = expf(f + m - mn);
        b[at] = expf(i - mn);
        em[at] = expf(-mn);
        m = mn;
    }
    if (t1 == T && t0 < t1) m_state[h] = m;                         // every thread has read m0 ahead of the barrier
}

// ---- recurrence over rows ----
// grid (ceil((vdim + 1) / COLS), heads, segments), 128 threads.  Lane l holds state elements W * (c LN + l) + j, c < CH, j < W, of each of its CB columns.
// PASS 0: the whole step, one segment.  The recurrence is linear once a and b are known, so a long step may be cut into segments of seg_len rows: the
// state behind a segment is (product of its a) * (state in front) + (state from zero).
// PASS 1: segments 0 .. segments - 2, state only: seg[z] <- the state from zero (segment 0: from the real one), decay[z] <- the product of the a;
//         segment 0 also keeps the step's first state in seg[last].
// PASS 2: every segment joins the states in front of it, then produces its rows; the last one writes the state back.
template <int LN, int CH, int W, int CB, int PASS>
__global__ void __launch_bounds__(128) mlstm_rows_kernel(float* __restrict__ out, float* __restrict__ den, const float* __restrict__ q, const float* __restrict__ k,
                                                         const float* __restrict__ v, const float* __restrict__ ga, const float* __restrict__ gb, float* __restrict__ state,
                                                         float q_scale, int T, int heads, int dim, int vdim, const int* __restrict__ pos_dev, int p0, float* __restrict__ seg,
                                                         float* __restrict__ decay, int seg_len, int segments) {
    constexpr int TILE = SCAN_TILE, THREADS = 128, COLS = THREADS / LN * CB, ROWS_LEFT = LN >= TILE ? 1 : TILE / LN;
    extern __shared__ __align__(16) float sm[];
    const int buf_floats = (2 * TILE * dim + TILE * COLS + 2 * TILE + 3) & ~3;      // q | k [TILE][dim], v [TILE][COLS], a | b [TILE]
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.y, n = heads * dim, nv = heads * vdim, all_cols = vdim + 1;
    const int col_l = threadIdx.x / LN * CB, l = threadIdx.x % LN;
    const int col = blockIdx.x * COLS + col_l;
    const bool fresh = (pos_dev ? *pos_dev : p0) == 0;
    const size_t all = (size_t)heads * all_cols * dim;
    auto st_off = [&](int b) { return ((size_t)h * all_cols + col + b) * dim; };       // only for live columns
    const int z = PASS == 0 ? 0 : blockIdx.z;
    if (PASS != 0) {                            // this segment's rows
        const size_t first = (size_t)z * seg_len;
        q += first * n; k += first * n; v += first * nv; ga += first * heads; gb += first * heads; out += first * nv; den += first * heads;
        T = min(seg_len, T - z * seg_len);
    }
    int d0[CH];
    bool on[CH];
    float S[CB][CH][W], prod = 1.f;
#pragma unroll
    for (int c = 0; c < CH; c++) {
        d0[c] = W * (c * LN + l);
        on[c] = d0[c] < dim;
#pragma unroll
        for (int b = 0; b < CB; b++) {
#pragma unroll
            for (int j = 0; j < W; j++) S[b][c][j] = 0.f;
            if (!on[c] || col + b >= all_cols) continue;
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
                    const float dy = decay[(size_t)y * heads + h];
#pragma unroll
                    for (int j = 0; j < W; j++) S[b][c][j] = fmaf(dy, S[b][c][j], seg[(size_t)y * all + at + j]);
                }
            }
        }
        if (!on[c]) d0[c] = 0;
    }
    auto load_tile = [&](int t0, int buf) {
        float* sq = sm + (size_t)buf * buf_floats;
        float* sk = sq + TILE * dim;
        float* sv = sk + TILE * dim;
        float* sa = sv + TILE * COLS;
        const int nt = min(TILE, T - t0), dv = dim / W;
        for (int i = threadIdx.x; i < nt * dv; i += THREADS) {
            const int tt = i / dv, d = (i - tt * dv) * W;
            const size_t at = (size_t)(t0 + tt) * n + (size_t)h * dim + d;
            if constexpr (W == 4) { if (PASS != 1) cp_async16(sq + tt * dim + d, q + at); cp_async16(sk + tt * dim + d, k + at); }
            else { if (PASS != 1) cp_async4(sq + tt * dim + d, q + at); cp_async4(sk + tt * dim + d, k + at); }
        }
        for (int i = threadIdx.x; i < nt * COLS; i += THREADS) {
            const int tt = i / COLS, c = blockIdx.x * COLS + i % COLS;
            if (c < vdim) cp_async4(sv + i, v + (size_t)(t0 + tt) * nv + (size_t)h * vdim + c);
            else sv[i] = c == vdim ? 1.f : 0.f;                     // the normalizer's value; columns past it stay zero
        }
        for (int i = threadIdx.x; i < nt; i += THREADS) { cp_async4(sa + i, ga + (size_t)(t0 + i) * heads + h); cp_async4(sa + TILE + i, gb + (size_t)(t0 + i) * heads + h); }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    const int n_tiles = (T + TILE - 1) / TILE;
    load_tile(0, 0);
    for (int x = 0; x < n_tiles; x++) {
        const int t0 = x * TILE, nt = min(TILE, T - t0), buf = x & 1;
        if (x + 1 < n_tiles) {
            load_tile(t0 + TILE, buf ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const float* sq = sm + (size_t)buf * buf_floats;
        const float* sk = sq + TILE * dim;
        const float* sv = sk + TILE * dim;
        const float* sa = sv + TILE * COLS;
        float part[CB][TILE];
        auto step = [&](int tt) {
            const float a = sa[tt], bg = sa[TILE + tt];
            float vj[CB], p[CB];
#pragma unroll
            for (int b = 0; b < CB; b++) { vj[b] = bg * sv[tt * COLS + col_l + b]; p[b] = 0.f; }
#pragma unroll
            for (int c = 0; c < CH; c++) {
                float qq[W], kk[W];
                if constexpr (W == 4) {
                    float4 e = make_float4(0.f, 0.f, 0.f, 0.f);
                    if (PASS != 1) e = ld4(sq + tt * dim + d0[c]);
                    const float4 g = ld4(sk + tt * dim + d0[c]);
                    qq[0] = e.x; qq[1] = e.y; qq[2] = e.z; qq[3] = e.w; kk[0] = g.x; kk[1] = g.y; kk[2] = g.z; kk[3] = g.w;
                } else { qq[0] = PASS != 1 ? sq[tt * dim + d0[c]] : 0.f; kk[0] = sk[tt * dim + d0[c]]; }
                if (CH == 1 || on[c]) {
#pragma unroll
                    for (int j = 0; j < W; j++) {
#pragma unroll
                        for (int b = 0; b < CB; b++) {
                            S[b][c][j] = fmaf(a, S[b][c][j], kk[j] * vj[b]);
                            if (PASS != 1) p[b] = fmaf(qq[j], S[b][c][j], p[b]);
                        }
                    }
                }
            }
            if (PASS == 1) prod *= a;
#pragma unroll
            for (int b = 0; b < CB; b++) part[b][tt] = (CH == 1 && !on[0]) ? 0.f : p[b];
        };
        if (nt == TILE) {
#pragma unroll
            for (int tt = 0; tt < TILE; tt++) step(tt);
        } else {
#pragma unroll
            for (int tt = 0; tt < TILE; tt++) {
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
                    if (tt >= nt || (LN > TILE && (l & 1) != 0)) continue;
                    if (col + b < vdim) out[(size_t)(t0 + tt) * nv + (size_t)h * vdim + col + b] = part[b][j] * q_scale;
                    else if (col + b == vdim) den[(size_t)(t0 + tt) * heads + h] = part[b][j] * q_scale;
                }
            }
        }
        __syncthreads();                       // the buffer is refilled by the load of tile x + 2
    }
    if (PASS == 2 && z != segments - 1) return;
    float* to = PASS == 1 ? seg + (size_t)z * all : state;
#pragma unroll
    for (int c = 0; c < CH; c++) {
        if (!on[c]) continue;
#pragma unroll
        for (int b = 0; b < CB; b++) {
            if (col + b >= all_cols) continue;
#pragma unroll
            for (int j = 0; j < W; j++) to[st_off(b) + d0[c] + j] = S[b][c][j];
        }
    }
    if (PASS == 1 && blockIdx.x == 0 && threadIdx.x == 0) decay[(size_t)z * heads + h] = prod;
}

// ---- quotient, head norm, output gate: a warp per (row, head) ----
// NV 16-byte pieces per lane; NV == 0: any width and alignment
template <int NV>
__global__ void __launch_bounds__(256) mlstm_out_norm_kernel(float* __restrict__ out, __nv_bfloat16* __restrict__ hi, size_t lo, const float* __restrict__ o,
                                                             const float* __restrict__ den, const float* __restrict__ em, const float* __restrict__ gate,
                                                             const float* __restrict__ norm, float eps, int items, int heads, int vdim) {
    pdl_launch_dependents();
    pdl_wait();
    const int th = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (th >= items) return;
    const int h = th % heads;
    const size_t base = (size_t)th * vdim;
    const float quot = 1.0f / (fmaxf(fabsf(den[th]), em[th]) + kDenEps);
    const float* nh = norm + (size_t)h * vdim;
    float ss = 0.f;
    if constexpr (NV > 0) {
        float4 v[NV];
#pragma unroll
        for (int i = 0; i < NV; i++) {
            const int d = 4 * (lane + 32 * i);
            v[i] = d < vdim ? ld4(o + base + d) : make_float4(0.f, 0.f, 0.f, 0.f);
            v[i].x *= quot; v[i].y *= quot; v[i].z *= quot; v[i].w *= quot;
            ss = fmaf(v[i].x, v[i].x, ss); ss = fmaf(v[i].y, v[i].y, ss); ss = fmaf(v[i].z, v[i].z, ss); ss = fmaf(v[i].w, v[i].w, ss);
        }
#pragma unroll
        for (int s = 16; s > 0; s >>= 1) ss += __shfl_xor_sync(0xFFFFFFFFu, ss, s);
        const float inv = 1.0f / sqrtf(ss / (float)vdim + eps);
#pragma unroll
        for (int i = 0; i < NV; i++) {
            const int d = 4 * (lane + 32 * i);
            if (d >= vdim) continue;
            const float4 N = ld4(nh + d), G = ld4(gate + base + d);
            const float y[4] = {v[i].x * inv * N.x * sigmoid_f(G.x), v[i].y * inv * N.y * sigmoid_f(G.y), v[i].z * inv * N.z * sigmoid_f(G.z), v[i].w * inv * N.w * sigmoid_f(G.w)};
            if (out) *reinterpret_cast<float4*>(out + base + d) = make_float4(y[0], y[1], y[2], y[3]);
            if (hi) split_store4(hi, hi + lo, base + d, y);
        }
    } else {
        for (int d = lane; d < vdim; d += 32) { const float y = o[base + d] * quot; ss = fmaf(y, y, ss); }
#pragma unroll
        for (int s = 16; s > 0; s >>= 1) ss += __shfl_xor_sync(0xFFFFFFFFu, ss, s);
        const float inv = 1.0f / sqrtf(ss / (float)vdim + eps);
        for (int d = lane; d < vdim; d += 32) {
            const float y = o[base + d] * quot * inv * nh[d] * sigmoid_f(gate[base + d]);
            if (out) out[base + d] = y;
            if (hi) split_store1(hi, hi + lo, base + d, y);
        }
    }
}

// ---- one token ----
// grid (splits, heads), the splits of a head form a cluster; 256 threads.  8 lanes per value channel; DV > 0: dim is a multiple of 4 and at most 32 DV, a
// lane's share of a channel is DV 16-byte pieces loaded together; DV == 0: any dim.  Every CTA works out the gates and <n, q> of its head; the first one
// replaces n and m once the cluster has read them.
constexpr int MT_LN = 8, MT_MAX_SPLITS = 8;
template <int DV>
__global__ void __launch_bounds__(256) mlstm_token_kernel(float* __restrict__ out, const float* __restrict__ q, const float* __restrict__ k, const float* __restrict__ v,
                                                          const float* __restrict__ gate, const float* __restrict__ zi, const float* __restrict__ zf, const float* __restrict__ bi,
                                                          const float* __restrict__ bf, const float* __restrict__ norm, float* __restrict__ state, float* __restrict__ m_state,
                                                          float cap, float q_scale, float eps, int dim, int vdim, const int* __restrict__ pos_dev, int p0) {
    namespace cg = cooperative_groups;
    extern __shared__ __align__(16) float sm[];
    const int dp = (dim + 3) & ~3, splits = gridDim.x, rank = blockIdx.x, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int per = (vdim + splits - 1) / splits, j_first = min(vdim, rank * per), j_end = min(vdim, j_first + per);
    float *qs = sm, *ks = qs + dp, *ns = ks + dp, *os = ns + dp;      // q, k, the new n [dim]; this CTA's channels [per]
    __shared__ float red[8];
    __shared__ float sq_sum;
    const size_t hs = (size_t)h * (vdim + 1) * dim, hq = (size_t)h * dim, hv = (size_t)h * vdim;
    // the state and the constants are older than this step: their way from HBM overlaps the projections
    l2_prefetch(state + hs + (size_t)j_first * dim, (size_t)(j_end - j_first) * dim * sizeof(float), threadIdx.x, 256);
    l2_prefetch(state + hs + (size_t)vdim * dim, (size_t)dim * sizeof(float), threadIdx.x, 256);
    l2_prefetch(norm + hv + j_first, (size_t)(j_end - j_first) * sizeof(float), threadIdx.x, 256);
    pdl_launch_dependents();
    pdl_wait();
    const bool fresh = (pos_dev ? *pos_dev : p0) == 0;
    const float m0 = fresh ? 0.f : m_state[h];
    const float gi = capped(zi[h] + bi[h], cap), gf = log_sigmoid(capped(zf[h] + bf[h], cap));
    const float m1 = fmaxf(gf + m0, gi), a = expf(gf + m0 - m1), b = expf(gi - m1);
    float nq = 0.f;
    for (int d = threadIdx.x; d < dim; d += 256) {
        const float qd = q[hq + d] * q_scale, kd = k[hq + d];
        qs[d] = qd; ks[d] = kd;
        const float nd = fmaf(a, fresh ? 0.f : state[hs + (size_t)vdim * dim + d], b * kd);
        ns[d] = nd;
        nq = fmaf(nd, qd, nq);
    }
#pragma unroll
    for (int s = 16; s > 0; s >>= 1) nq += __shfl_xor_sync(0xFFFFFFFFu, nq, s);
    if (lane == 0) red[warp] = nq;
    __syncthreads();
    nq = 0.f;
#pragma unroll
    for (int w = 0; w < 8; w++) nq += red[w];
    const float quot = 1.0f / (fmaxf(fabsf(nq), expf(-m1)) + kDenEps);
    const int l = threadIdx.x % MT_LN;
#pragma unroll 2
    for (int j0 = j_first; j0 < j_end; j0 += 256 / MT_LN) {
        const int j = j0 + threadIdx.x / MT_LN;
        const bool live = j < j_end;
        float* st = state + hs + (size_t)(live ? j : j_first) * dim;
        const float vj = live ? b * v[hv + j] : 0.f;
        float p = 0.f;
        if constexpr (DV > 0) {
            float4 S[DV];
#pragma unroll
            for (int c = 0; c < DV; c++) {
                const int d = 4 * (c * MT_LN + l);
                S[c] = (live && !fresh && d < dim) ? ld4(st + d) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
#pragma unroll
            for (int c = 0; c < DV; c++) {
                const int d = 4 * (c * MT_LN + l);
                if (live && d < dim) {
                    const float4 Q = ld4(qs + d), K = ld4(ks + d);
                    S[c].x = fmaf(a, S[c].x, K.x * vj); S[c].y = fmaf(a, S[c].y, K.y * vj); S[c].z = fmaf(a, S[c].z, K.z * vj); S[c].w = fmaf(a, S[c].w, K.w * vj);
                    p = fmaf(Q.x, S[c].x, p); p = fmaf(Q.y, S[c].y, p); p = fmaf(Q.z, S[c].z, p); p = fmaf(Q.w, S[c].w, p);
                    *reinterpret_cast<float4*>(st + d) = S[c];
                }
            }
        } else {
            for (int d = l; live && d < dim; d += MT_LN) {
                const float S = fmaf(a, fresh ? 0.f : st[d], ks[d] * vj);
                p = fmaf(qs[d], S, p);
                st[d] = S;
            }
        }
#pragma unroll
        for (int s = MT_LN / 2; s > 0; s >>= 1) p += __shfl_xor_sync(0xFFFFFFFFu, p, s);
        if (l == 0 && live) os[j - j_first] = p * quot;
    }
    __syncthreads();
    float ss = 0.f;
    for (int j = threadIdx.x; j < j_end - j_first; j += 256) ss = fmaf(os[j], os[j], ss);
#pragma unroll
    for (int s = 16; s > 0; s >>= 1) ss += __shfl_xor_sync(0xFFFFFFFFu, ss, s);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int w = 0; w < 8; w++) tot += red[w];
    if (splits > 1) {
        cg::cluster_group cluster = cg::this_cluster();
        if (threadIdx.x == 0) sq_sum = tot;
        cluster.sync();
        tot = 0.f;
        for (int r = 0; r < splits; r++) tot += *cluster.map_shared_rank(&sq_sum, r);
        cluster.sync();                          // no CTA leaves while another one reads its sum; n and m have been read by all
    }
    if (rank == 0) {
        for (int d = threadIdx.x; d < dim; d += 256) state[hs + (size_t)vdim * dim + d] = ns[d];
        if (threadIdx.x == 0) m_state[h] = m1;
    }
    const float inv = 1.0f / sqrtf(tot / (float)vdim + eps);
    for (int j = j_first + threadIdx.x; j < j_end; j += 256) out[hv + j] = os[j - j_first] * inv * norm[hv + j] * sigmoid_f(gate[hv + j]);
}

constexpr int MR_MAX_SEGMENTS = 16;
template <int LN, int CH, int W, int CB>
void launch_rows(float* o, float* den, const float* q, const float* k, const float* v, const float* a, const float* b, float* state, float q_scale, int T, int heads, int dim,
                 int vdim, const int* pos_dev, int p0, float* scratch, cudaStream_t s) {
    constexpr int COLS = 128 / LN * CB;
    const size_t buf = ((size_t)2 * SCAN_TILE * dim + (size_t)SCAN_TILE * COLS + 2 * SCAN_TILE + 3) & ~(size_t)3;
    const size_t smem = sizeof(float) * 2 * buf;
    NT_CHECK(smem <= 200 * 1024, "mlstm_rows: the tiles do not fit in shared memory");
    const int cols = (vdim + 1 + COLS - 1) / COLS;
    // segments where the columns leave SMs without a CTA or with one only: until about four CTAs stand on every SM, none shorter than eight tiles.
    // The state pass costs about half of a full one, so two segments gain nothing.
    int segments = 1;
    if (scratch && cols * heads <= 148) segments = std::max(1, std::min({MR_MAX_SEGMENTS, (4 * 148 + cols * heads - 1) / (cols * heads), T / (8 * SCAN_TILE)}));
    if (segments < 3) segments = 1;
    const int seg_len = ((T + segments - 1) / segments + SCAN_TILE - 1) / SCAN_TILE * SCAN_TILE;
    segments = (T + seg_len - 1) / seg_len;
    static unsigned long long done0 = 0, done1 = 0, done2 = 0;
    if (segments == 1) {
        if (smem > 48 * 1024) opt_in_dynamic_smem(mlstm_rows_kernel<LN, CH, W, CB, 0>, 200 * 1024, done0);
        launch_k(mlstm_rows_kernel<LN, CH, W, CB, 0>, dim3(cols, heads), dim3(128), smem, s, o, den, q, k, v, a, b, state, q_scale, T, heads, dim, vdim, pos_dev, p0, (float*)nullptr,
                 (float*)nullptr, T, 1);
        count_launch();
        return;
    }
    float* decay = scratch + (size_t)MR_MAX_SEGMENTS * heads * ((size_t)vdim + 1) * dim;
    if (smem > 48 * 1024) { opt_in_dynamic_smem(mlstm_rows_kernel<LN, CH, W, CB, 1>, 200 * 1024, done1); opt_in_dynamic_smem(mlstm_rows_kernel<LN, CH, W, CB, 2>, 200 * 1024, done2); }
    launch_k(mlstm_rows_kernel<LN, CH, W, CB, 1>, dim3(cols, heads, segments - 1), dim3(128), smem, s, o, den, q, k, v, a, b, state, q_scale, T, heads, dim, vdim, pos_dev, p0, scratch,
             decay, seg_len, segments);
    launch_k(mlstm_rows_kernel<LN, CH, W, CB, 2>, dim3(cols, heads, segments), dim3(128), smem, s, o, den, q, k, v, a, b, state, q_scale, T, heads, dim, vdim, pos_dev, p0, scratch, decay,
             seg_len, segments);
    count_launch(2);
}

bool aligned16(std::initializer_list<const void*> ps) {
    uintptr_t bits = 0;
    for (const void* p : ps) bits |= reinterpret_cast<uintptr_t>(p);
    return (bits & 15) == 0;
}

}  // namespace

void mlstm_gates(float* a, float* b, float* em, const float* zi, const float* zf, int ld, const float* bi, const float* bf, float cap, float* m, int T, int heads,
                 const int* pos_dev, int p0, cudaStream_t s) {
    if (T <= 0) return;
    NT_CHECK(cap > 0.f, "mlstm_gates: the gates' cap must be positive");
    launch_k(mlstm_gates_kernel, dim3(heads), dim3(GT_THREADS), 0, s, a, b, em, zi, zf, ld, bi, bf, cap, m, T, heads, pos_dev, p0);
    count_launch();
}

size_t mlstm_rows_scratch_floats(int heads, int dim, int vdim) { return (size_t)MR_MAX_SEGMENTS * heads * (((size_t)vdim + 1) * dim + 1); }

void mlstm_rows(float* o, float* den, const float* q, const float* k, const float* v, const float* a, const float* b, float* state, float q_scale, int T, int heads, int dim,
                int vdim, const int* pos_dev, int p0, cudaStream_t s, float* scratch) {
    NT_CHECK(dim >= 1 && dim <= MLSTM_MAX_DIM && vdim >= 1, "mlstm_rows: query / key heads wider than 512 are not covered");
    if (T <= 0) return;
#define NT_MR(LN, CH, W, CB) launch_rows<LN, CH, W, CB>(o, den, q, k, v, a, b, state, q_scale, T, heads, dim, vdim, pos_dev, p0, scratch, s)
    if (dim % 4 == 0 && aligned16({q, k})) {
        if (dim <= 16) NT_MR(4, 1, 4, 1);
        else if (dim <= 32) NT_MR(8, 1, 4, 2);
        else if (dim <= 64) NT_MR(16, 1, 4, 4);
        else if (dim <= 128) NT_MR(32, 1, 4, 4);
        else if (dim <= 256) NT_MR(32, 2, 4, 4);
        else NT_MR(32, 4, 4, 2);
    } else {
        if (dim <= 8) NT_MR(8, 1, 1, 1);
        else if (dim <= 32) NT_MR(16, 2, 1, 1);
        else if (dim <= 128) NT_MR(16, 8, 1, 1);
        else NT_MR(32, 16, 1, 1);
    }
#undef NT_MR
}

void mlstm_out_norm(float* out, void* split, const float* o, const float* den, const float* em, const float* gate, const float* norm, float eps, int T, int heads, int vdim,
                    cudaStream_t s) {
    const int items = T * heads;
    if (items <= 0) return;
    const dim3 grid((items + 7) / 8);
#define NT_MN(NV) launch_k(mlstm_out_norm_kernel<NV>, grid, dim3(256), 0, s, out, static_cast<__nv_bfloat16*>(split), split_lo_offset(T, heads * vdim), o, den, em, gate, norm, eps, items, \
                           heads, vdim)
    if (vdim % 4 == 0 && vdim <= 512 && aligned16({out, split, o, gate, norm})) { if (vdim <= 128) NT_MN(1); else if (vdim <= 256) NT_MN(2); else NT_MN(4); }
    else NT_MN(0);
#undef NT_MN
    count_launch();
}

void mlstm_token(float* out, const float* q, const float* k, const float* v, const float* gate, const float* zi, const float* zf, const float* bi, const float* bf,
                 const float* norm, float* state, float* m, float cap, float q_scale, float eps, int heads, int dim, int vdim, const int* pos_dev, int p0, cudaStream_t s) {
    NT_CHECK(dim >= 1 && dim <= MLSTM_MAX_DIM && vdim >= 1 && cap > 0.f, "mlstm_token: query / key heads wider than 512 are not covered");
    // a head's channels over up to 8 CTAs, 32 channels (one pass of the CTA) or more each
    int splits = 1;
    while (splits < MT_MAX_SPLITS && splits * heads < 148 && vdim >= 64 * splits) splits *= 2;
    const int per = (vdim + splits - 1) / splits;
    const size_t smem = sizeof(float) * (3 * (size_t)((dim + 3) & ~3) + (size_t)per);
    NT_CHECK(smem <= 47 * 1024, "mlstm_token: the head does not fit in shared memory");
    const int dv = dim % 4 || !aligned16({state}) ? 0 : dim <= 32 ? 1 : dim <= 64 ? 2 : dim <= 128 ? 4 : dim <= 256 ? 8 : 16;
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = dim3(splits, heads); cfg.blockDim = dim3(256); cfg.dynamicSmemBytes = smem; cfg.stream = s;
    cudaLaunchAttribute at[2];
    at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[0].val.programmaticStreamSerializationAllowed = pdl_enabled() ? 1 : 0;
    at[1].id = cudaLaunchAttributeClusterDimension;
    at[1].val.clusterDim.x = (unsigned)splits; at[1].val.clusterDim.y = 1; at[1].val.clusterDim.z = 1;
    cfg.attrs = at; cfg.numAttrs = 2;
    auto* kern = dv == 1 ? mlstm_token_kernel<1> : dv == 2 ? mlstm_token_kernel<2> : dv == 4 ? mlstm_token_kernel<4> : dv == 8 ? mlstm_token_kernel<8> : dv == 16 ? mlstm_token_kernel<16>
                                                                                                                                                            : mlstm_token_kernel<0>;
    NT_CUDA_CHECK(cudaLaunchKernelEx(&cfg, kern, out, q, k, v, gate, zi, zf, bi, bf, norm, state, m, cap, q_scale, eps, dim, vdim, pos_dev, p0));
    count_launch();
}

}}  // namespace nt::b200
