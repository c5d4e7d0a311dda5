// attention_rows_decode.cu — attention of ONE query token over BF16 cache rows, for query heads that share key / value heads: grouped-query attention
// (heads / kv_heads query heads per key head, keys and values in rows of their own) and the absorbed form of the latent attention (all heads over one
// row per position whose first vdim numbers are the values).
//       s_hj = scale <q_h, k_j> - slope_h (pos - j),   j <= pos  (window > 0: only the last `window` positions)
// A CTA owns (a slice of the visible positions, one key / value head) and serves every query head of that key head from one shared-memory copy of the
// rows: tiles of 64 positions by cp.async, the queries as BF16 hi / lo pairs, scores and weighted sums on the warp-level tensor-core path (mma.sync
// m16n8k16, F32 accumulate: 16 or 32 heads are one or two row tiles, shorter groups leave rows unused), softmax weights split into hi / lo pairs as in
// attention_prefill_mma.cu.  Score tile: a warp per 8 positions.  Weighted sum: a warp per 16 value channels, 16 positions per step.
// Every CTA writes (max, sum, unnormalised vector) per head; the merge kernels (attention_latent.cu) join the slices.
// The grid depends on the cache's length only, never on the position: the captured decode step replays it unchanged.
// Compiled WITHOUT --use_fast_math.
#include "kernels_internal.h"
#include "bf16_split.cuh"
#include "ring.cuh"
#include <cuda_bf16.h>
#include <algorithm>
#include <cfloat>
#include <cstdlib>

namespace nt { namespace b200 {

namespace {

constexpr int TK = ROWS_DECODE_TILE, LDS = TK + 4, LDP = TK + 8;      // positions per tile; row strides of the score and weight tiles
constexpr int MAX_PAIRS = 4;                                          // 16-channel pieces per warp: vdim <= 512

__device__ __forceinline__ uint32_t smem_at(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp16(void* dst, const void* src) { asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_at(dst)), "l"(src) : "memory"); }
__device__ __forceinline__ void mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_at(p)));
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_at(p)));
}
__device__ __forceinline__ void ldsm2(uint32_t (&r)[2], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0, %1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(smem_at(p)));
}

size_t smem_bytes(int mt, int dim, int vdim, bool same) {
    const size_t rows = 16 * (size_t)mt;
    return 2 * rows * (dim + 8) * 2 + (size_t)TK * (dim + 8) * 2 + (same ? 0 : (size_t)TK * (vdim + 8) * 2) + rows * LDS * 4 + 2 * rows * LDP * 2 + rows * 4;
}

// grid (slices, kv_heads), 256 threads.  MT: row tiles of 16 query heads.
template <int MT>
__global__ void __launch_bounds__(256) rows_decode_kernel(float* __restrict__ part, const float* __restrict__ Q, const __nv_bfloat16* __restrict__ kc, const __nv_bfloat16* __restrict__ vc,
                                                          const int* __restrict__ pos_dev, int p0, int heads, int kv_heads, int dim, int vdim, int k_stride, int v_stride, float scale,
                                                          int window, const float* __restrict__ slopes, int same) {
    constexpr int ROWS = 16 * MT, TPR = 256 / ROWS, KPT = TK / TPR;        // threads per row and positions per thread in the softmax
    extern __shared__ __align__(16) unsigned char raw[];
    const int ldq = dim + 8, ldv = same ? ldq : vdim + 8, group = heads / kv_heads, g0 = blockIdx.y;
    __nv_bfloat16* qh = reinterpret_cast<__nv_bfloat16*>(raw);             // [ROWS][ldq]
    __nv_bfloat16* ql = qh + (size_t)ROWS * ldq;
    __nv_bfloat16* kt = ql + (size_t)ROWS * ldq;                           // [TK][ldq]
    __nv_bfloat16* vt = same ? kt : kt + (size_t)TK * ldq;                 // [TK][ldv]
    float* ss = reinterpret_cast<float*>(kt + (size_t)TK * ldq + (same ? 0 : (size_t)TK * ldv));      // [ROWS][LDS]
    __nv_bfloat16* ph = reinterpret_cast<__nv_bfloat16*>(ss + ROWS * LDS); // [ROWS][LDP]
    __nv_bfloat16* pl = ph + ROWS * LDP;
    float* corr_s = reinterpret_cast<float*>(pl + ROWS * LDP);             // [ROWS]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, slice = blockIdx.x, n_slices = gridDim.x;
    pdl_launch_dependents();
    pdl_wait();
    const int pos = pos_dev ? *pos_dev : p0, lo = window > 0 ? max(0, pos + 1 - window) : 0, n_vis = pos + 1 - lo;
    auto load_tile = [&](int t0) {
        const int ck = dim / 8, cv = vdim / 8;
        // 8 or 32 lanes per row: no division, whole sectors
        const int lanes = ck <= 16 ? 8 : 32, l0 = threadIdx.x & (lanes - 1), rows_at_once = 256 / lanes;
        for (int r = threadIdx.x / lanes; r < TK; r += rows_at_once) {
            const int j = lo + min(t0 + r, n_vis - 1);                         // rows past the last visible one are masked below
            const __nv_bfloat16* src = kc + (size_t)j * k_stride + (size_t)g0 * dim;
            for (int c = l0; c < ck; c += lanes) cp16(kt + (size_t)r * ldq + c * 8, src + c * 8);
            if (!same) {
                const __nv_bfloat16* vs = vc + (size_t)j * v_stride + (size_t)g0 * vdim;
                for (int c = l0; c < cv; c += lanes) cp16(vt + (size_t)r * ldv + c * 8, vs + c * 8);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    int t0 = slice * TK;
    if (t0 < n_vis) load_tile(t0);
    if (t0 < n_vis)
        for (int r = warp; r < ROWS; r += 8) {
            const float* q = Q + ((size_t)g0 * group + r) * dim;
#pragma unroll 2
            for (int c = lane * 4; c < dim; c += 128) {
                float v[4] = {0.f, 0.f, 0.f, 0.f};
                if (r < group) { const float4 f = *reinterpret_cast<const float4*>(q + c); v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w; }
                split_store4(qh, ql, (size_t)r * ldq + c, v);
            }
        }
    const int srow = threadIdx.x / TPR, sl = threadIdx.x % TPR;
    const float slope = slopes && srow < group ? slopes[g0 * group + srow] : 0.f;
    float m = -FLT_MAX, l = 0.f, o[MT][MAX_PAIRS][2][4];
#pragma unroll
    for (int a = 0; a < MT; a++)
#pragma unroll
        for (int b = 0; b < MAX_PAIRS; b++)
#pragma unroll
            for (int e = 0; e < 4; e++) o[a][b][0][e] = o[a][b][1][e] = 0.f;
    const int pairs = vdim / 16;
    for (; t0 < n_vis; t0 += n_slices * TK) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        // ---- scores: 8 positions per warp, hi and lo products in chains of their own ----
        float sh[MT][4], sl4[MT][4];
#pragma unroll
        for (int a = 0; a < MT; a++)
#pragma unroll
            for (int e = 0; e < 4; e++) sh[a][e] = sl4[a][e] = 0.f;
#pragma unroll 4
        for (int ks = 0; ks < dim / 16; ks++) {
            uint32_t b[2];
            ldsm2(b, kt + (size_t)(warp * 8 + (lane & 7)) * ldq + ks * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
            for (int a = 0; a < MT; a++) {
                uint32_t ah[4], al[4];
                const size_t at = (size_t)(a * 16 + (lane & 15)) * ldq + ks * 16 + (lane >> 4) * 8;
                ldsm4(ah, qh + at);
                ldsm4(al, ql + at);
                mma(sh[a], ah, b[0], b[1]);
                mma(sl4[a], al, b[0], b[1]);
            }
        }
#pragma unroll
        for (int a = 0; a < MT; a++) {
            float* d = ss + (a * 16 + (lane >> 2)) * LDS + warp * 8 + 2 * (lane & 3);
            *reinterpret_cast<float2*>(d) = make_float2(sh[a][0] + sl4[a][0], sh[a][1] + sl4[a][1]);
            *reinterpret_cast<float2*>(d + 8 * LDS) = make_float2(sh[a][2] + sl4[a][2], sh[a][3] + sl4[a][3]);
        }
        __syncthreads();
        // ---- softmax: TPR threads per head ----
        float s[KPT], mx = -FLT_MAX;
#pragma unroll
        for (int e = 0; e < KPT; e++) {
            const int j = t0 + sl + e * TPR;                               // position lo + j
            s[e] = j < n_vis ? ss[srow * LDS + sl + e * TPR] * scale - slope * (float)(pos - (lo + j)) : -FLT_MAX;
            mx = fmaxf(mx, s[e]);
        }
#pragma unroll
        for (int q = TPR / 2; q > 0; q >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xFFFFFFFFu, mx, q));
        const float mn = fmaxf(m, mx), corr = expf(m - mn);
        float sum = 0.f;
#pragma unroll
        for (int e = 0; e < KPT; e++) {
            const float pk = t0 + sl + e * TPR < n_vis ? expf(s[e] - mn) : 0.f;
            sum += pk;
            const __nv_bfloat16 hb = __float2bfloat16_rn(pk);
            ph[srow * LDP + sl + e * TPR] = hb;
            pl[srow * LDP + sl + e * TPR] = __float2bfloat16_rn(pk - __bfloat162float(hb));
        }
#pragma unroll
        for (int q = TPR / 2; q > 0; q >>= 1) sum += __shfl_xor_sync(0xFFFFFFFFu, sum, q);
        l = l * corr + sum;
        m = mn;
        if (sl == 0) corr_s[srow] = corr;
        __syncthreads();
        // ---- weighted sum: 16 channels per warp and piece ----
#pragma unroll
        for (int a = 0; a < MT; a++) {
            const float c0 = corr_s[a * 16 + (lane >> 2)], c1 = corr_s[a * 16 + 8 + (lane >> 2)];
#pragma unroll
            for (int b = 0; b < MAX_PAIRS; b++)
#pragma unroll
                for (int n = 0; n < 2; n++) { o[a][b][n][0] *= c0; o[a][b][n][1] *= c0; o[a][b][n][2] *= c1; o[a][b][n][3] *= c1; }
        }
#pragma unroll
        for (int k16 = 0; k16 < TK / 16; k16++) {
            uint32_t ah[MT][4], al[MT][4];
#pragma unroll
            for (int a = 0; a < MT; a++) {
                const int at = (a * 16 + (lane & 15)) * LDP + k16 * 16 + (lane >> 4) * 8;
                ldsm4(ah[a], ph + at);
                ldsm4(al[a], pl + at);
            }
#pragma unroll
            for (int b = 0; b < MAX_PAIRS; b++) {
                const int np = warp + 8 * b;
                if (np >= pairs) continue;                                 // uniform in the warp
                uint32_t v[4];
                ldsm4t(v, vt + (size_t)(k16 * 16 + (lane & 15)) * ldv + np * 16 + (lane >> 4) * 8);
#pragma unroll
                for (int a = 0; a < MT; a++) {
                    mma(o[a][b][0], ah[a], v[0], v[1]);
                    mma(o[a][b][1], ah[a], v[2], v[3]);
                    mma(o[a][b][0], al[a], v[0], v[1]);
                    mma(o[a][b][1], al[a], v[2], v[3]);
                }
            }
        }
        __syncthreads();                                                   // the tile is consumed
        if (t0 + n_slices * TK < n_vis) load_tile(t0 + n_slices * TK);
    }
    auto dst_of = [&](int r) { return part + ((size_t)slice * heads + (size_t)g0 * group + r) * (vdim + 2); };
    if (sl == 0 && srow < group) { float* d = dst_of(srow); d[0] = m; d[1] = l; }
#pragma unroll
    for (int a = 0; a < MT; a++)
#pragma unroll
        for (int b = 0; b < MAX_PAIRS; b++) {
            const int np = warp + 8 * b;
            if (np >= pairs) continue;
#pragma unroll
            for (int n = 0; n < 2; n++) {
                const int c = np * 16 + n * 8 + 2 * (lane & 3), r0 = a * 16 + (lane >> 2), r1 = r0 + 8;
                if (r0 < group) { float* d = dst_of(r0) + 2 + c; d[0] = o[a][b][n][0]; d[1] = o[a][b][n][1]; }
                if (r1 < group) { float* d = dst_of(r1) + 2 + c; d[0] = o[a][b][n][2]; d[1] = o[a][b][n][3]; }
            }
        }
}

}  // namespace

bool attention_rows_decode_supported(int heads, int kv_heads, int dim, int vdim, int k_stride, int v_stride, DType cache_dt, const void* k, const void* v) {
    static const bool off = getenv("NT_B200_NO_ROWS_DECODE") != nullptr;
    if (off || cache_dt != DType::BF16 || kv_heads < 1 || heads % kv_heads || dim < 16 || vdim < 16) return false;
    const int group = heads / kv_heads;
    return group <= 32 && dim % 16 == 0 && vdim % 16 == 0 && vdim <= 128 * MAX_PAIRS && k_stride % 8 == 0 && v_stride % 8 == 0 && (k != v || vdim <= dim) &&
           ((reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v)) & 15) == 0 && smem_bytes(group > 16 ? 2 : 1, dim, vdim, k == v) <= 200 * 1024;
}
int attention_rows_decode_slices(int max_seq, int kv_heads, int window) {
    const int longest = window > 0 ? std::min(max_seq, window) : max_seq;
    return std::max(1, std::min((longest + TK - 1) / TK, ROWS_DECODE_MAX_SLICES / std::max(1, std::min(kv_heads, ROWS_DECODE_MAX_SLICES))));
}
size_t attention_rows_decode_scratch_floats(int heads, int vdim) { return (size_t)ROWS_DECODE_MAX_SLICES * heads * ((size_t)vdim + 2); }

int attention_rows_decode(float* part, const float* Q, const void* k, const void* v, const int* pos_dev, int p0, int max_seq, int heads, int kv_heads, int dim, int vdim, int k_stride,
                          int v_stride, float scale, int window, const float* slopes, cudaStream_t s) {
    NT_CHECK(attention_rows_decode_supported(heads, kv_heads, dim, vdim, k_stride, v_stride, DType::BF16, k, v), "attention_rows_decode: shape not covered");
    NT_CHECK((reinterpret_cast<uintptr_t>(Q) & 15) == 0, "attention_rows_decode: the queries must start on 16 bytes");
    const int mt = heads / kv_heads > 16 ? 2 : 1, slices = attention_rows_decode_slices(max_seq, kv_heads, window);
    const size_t smem = smem_bytes(mt, dim, vdim, k == v);
    const __nv_bfloat16 *kb = static_cast<const __nv_bfloat16*>(k), *vb = static_cast<const __nv_bfloat16*>(v);
    static unsigned long long done1 = 0, done2 = 0;
#define NT_RD(MT, DONE) { if (smem > 48 * 1024) opt_in_dynamic_smem(rows_decode_kernel<MT>, 200 * 1024, DONE); \
                          launch_k(rows_decode_kernel<MT>, dim3(slices, kv_heads), dim3(256), smem, s, part, Q, kb, vb, pos_dev, p0, heads, kv_heads, dim, vdim, k_stride, v_stride, scale, \
                                   window, slopes, k == v ? 1 : 0); }
    if (mt == 1) NT_RD(1, done1) else NT_RD(2, done2)
#undef NT_RD
    count_launch();
    return slices;
}

}}  // namespace nt::b200
