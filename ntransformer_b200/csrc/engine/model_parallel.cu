// model_parallel.cu — layers of BlockForm::PARALLEL whose mixer is the latent attention or the WKV time mixer, for the resident
// layer-spec model (engine/model_spec.cu).  Per layer, with n() the grouped RMS norm:
//       h = n(x_i, g);   X_(i+1) = x_i + mixer(h) + ff(h);   x_(i+1) = sum_j w_i[j] X_j,  j = 0 .. i + 1   (X_0: the embedding output)
// The results X_j of a step's rows live in slots [layers + 1][rows, width].  Slot i + 1 starts as x_i — the launch that averages the depth
// writes it there — and the last products of mixer and feed-forward are added in place, so X_(i+1) needs no copy and no sum of its own.
//
// One decoded token, 4 launches for a WKV layer with a dense feed-forward:
//   [depth average + grouped norm + the five shift blends]  [r, k, v, gate, tanh(W_w1 .) and xielu(W_up .): one launch, an input per matrix]
//   [decay, recurrence, head norm, gate]  [slot += W_o o + W_down a]
// and 9 for a latent-attention layer with routed experts:
//   [depth average + grouped norm]  [q, key / value latent, router logits]  [latent norm, rotation, cache write]  [absorbed queries]
//   [attention over the window's rows] [merge]  [values]  [choice + experts and shared expert up]  [slot += W_o o + experts + shared expert].
// Prompt rows take the tensor-core GEMMs (residual added in the epilogue), the tiled window attention over expanded rows and the tiled
// recurrence.  What a sequence carries between steps — cache rows, the WKV state, its previous mixer input, the previous token — is
// written by the step that owns the tokens and read by later steps only from there; every state reads as zeros when a step starts at
// position 0, so a new request needs no clearing.
#include "model.h"

#include <algorithm>
#include <cmath>

namespace nt { namespace b200 {

namespace {
template <typename T> T* dmalloc0(size_t n) {
    T* p = nullptr;
    NT_CUDA_CHECK(cudaMalloc(&p, std::max<size_t>(n, 1) * sizeof(T)));
    NT_CUDA_CHECK(cudaMemset(p, 0, std::max<size_t>(n, 1) * sizeof(T)));
    return p;
}
constexpr size_t kSlack = 64;                     // floats behind a layer's intermediates for the 16-byte alignment of the buffers carved from them
size_t up4(size_t n) { return (n + 3) & ~(size_t)3; }
MultiMat multi(const Weight& w, const float* x, float* y, GemvAct act = GEMV_ACT_NONE, const float* act_p = nullptr) {
    MultiMat m;
    m.W = w.ptr; m.dtype = w.dtype; m.row_pitch = w.pitch; m.x = x; m.y = y; m.out = w.rows; m.K = w.cols; m.act = act; m.act_p = act_p;
    return m;
}
// floats per row of a layer's intermediates: the decode step's and the prompt pass's layouts both fit
size_t layer_floats(const LayerSpec& S, size_t width) {
    const size_t H = (size_t)S.heads, D = (size_t)S.dim;
    size_t n = 0;
    if (S.mixer == MixerKind::WKV) n += 5 * width + 5 * H * D + (size_t)S.wkv.decay_rank + H + 2 * H * D;
    else {
        const size_t r = (size_t)S.latent.kv_rank, R = (size_t)S.latent.rot_dim;
        n += H * (D + R) + r + R + H * (r + R) + H * r + H * (size_t)S.vdim;
    }
    if (S.ff > 0 && S.ff_kind == FfKind::MLP) n += (size_t)S.ff;
    if (S.ff > 0 && S.ff_kind == FfKind::MOE_GLU) n += (size_t)S.experts + (size_t)S.top * S.ff + 3 * (size_t)S.shared_ff;
    return n;
}
}  // namespace

bool Model::parallel_rows() const { return cfg_.layers[0].form == BlockForm::PARALLEL && cfg_.layers[0].mixer != MixerKind::ATTN_WINDOW; }

bool Model::finalize_parallel_layer(int i) {
    const LayerSpec& S = cfg_.layers[(size_t)i];
    LayerWeights& M = layers_[(size_t)i];
    if (S.form != BlockForm::PARALLEL || S.weights_of >= 0 || S.layer_scale || S.kv_from >= 0 || cfg_.residual_mult != 1.f) {
        fprintf(stderr, "model: layer %d: this block form is not covered beside parallel latent-attention / WKV layers\n", i);
        return false;
    }
    if (cfg_.norm_groups > DENSE_MAX_NORM_GROUPS || cfg_.hidden_size % cfg_.norm_groups) { fprintf(stderr, "model: norm groups must divide the width (at most %d)\n", DENSE_MAX_NORM_GROUPS); return false; }
    bool ok = M.attn_norm && M.wo.ptr && (!cfg_.depth_average || M.depth_w) && (cfg_.bigram_buckets <= 0 || bigram_.ptr);
    std::vector<const Weight*> mats = {&M.wo};
    if (S.mixer == MixerKind::ATTN_LATENT) {
        if (S.latent.q_rank > 0) { fprintf(stderr, "model: layer %d: a query latent is not covered in the parallel block\n", i); return false; }
        if (S.latent.kv_rank > 512) { fprintf(stderr, "model: layer %d: latents wider than 512 are not covered\n", i); return false; }
        ok = ok && M.wq.ptr && M.w_dkv.ptr && M.dkv_norm && (S.dim == 0 || M.w_uk.ptr) && M.w_uv.ptr;
        mats.insert(mats.end(), {&M.wq, &M.w_dkv, &M.w_uv});
        if (S.dim > 0) mats.push_back(&M.w_uk);
    } else if (S.mixer == MixerKind::WKV) {
        if (S.dim > WKV_MAX_DIM) { fprintf(stderr, "model: layer %d: WKV heads wider than %d are not covered\n", i, WKV_MAX_DIM); return false; }
        for (const float* mu : M.wkv_mu) ok = ok && mu;
        ok = ok && M.wq.ptr && M.wk.ptr && M.wv.ptr && M.wkv_g.ptr && M.wkv_w1.ptr && M.wkv_w2.ptr && M.wkv_w0 && M.wkv_u && M.wkv_norm && S.wkv.decay_rank > 0;
        mats.insert(mats.end(), {&M.wq, &M.wk, &M.wv, &M.wkv_g, &M.wkv_w1, &M.wkv_w2});
    } else { fprintf(stderr, "model: layer %d: this mixer is not covered beside parallel latent-attention / WKV layers\n", i); return false; }
    if (S.ff > 0 && S.ff_kind == FfKind::MLP) {
        if (S.act != GluAct::XIELU || S.ff_bias) { fprintf(stderr, "model: layer %d: this feed-forward activation is not covered in the parallel block\n", i); return false; }
        ok = ok && M.up.ptr && M.down.ptr && M.ff_act;
        mats.insert(mats.end(), {&M.up, &M.down});
    } else if (S.ff > 0 && S.ff_kind == FfKind::MOE_GLU) {
        if (!S.route.all || S.act != GluAct::SILU || (S.shared_ff > 0 && !S.shared_glu)) { fprintf(stderr, "model: layer %d: this router is not covered in the parallel block\n", i); return false; }
        ok = ok && M.router && (int)M.e_up.size() == S.experts && (int)M.e_down.size() == S.experts && (int)M.e_gate.size() == S.experts;
        for (int e = 0; ok && e < S.experts; e++) mats.insert(mats.end(), {&M.e_up[(size_t)e], &M.e_down[(size_t)e], &M.e_gate[(size_t)e]});
        if (S.shared_ff > 0) mats.insert(mats.end(), {&M.sh_glu, &M.sh_up, &M.sh_down});
    } else if (S.ff > 0) { fprintf(stderr, "model: layer %d: this feed-forward is not covered in the parallel block\n", i); return false; }
    for (const Weight* w : mats) ok = ok && w->ptr;
    if (!ok) { fprintf(stderr, "model: layer %d is missing tensors\n", i); return false; }
    for (const Weight* w : mats)
        if (w->dtype != mats[0]->dtype || w->pitch != dtype_row_size(w->dtype, (size_t)w->cols)) { fprintf(stderr, "model: layer %d: its matrices must have one dtype and packed rows\n", i); return false; }
    if (S.mixer == MixerKind::WKV) {
        M.shift_state = dmalloc0<float>((size_t)cfg_.hidden_size);
        M.wkv_state = dmalloc0<float>((size_t)S.heads * S.dim * S.dim);
        for (Weight* w : {&M.wq, &M.wk, &M.wv, &M.wkv_g, &M.wkv_w1}) pad_for_tensor_cores(*w);
    } else for (Weight* w : {&M.wq, &M.w_dkv}) pad_for_tensor_cores(*w);
    if (S.ff > 0 && S.ff_kind == FfKind::MLP) pad_for_tensor_cores(M.up);
    if (S.ff > 0 && S.ff_kind == FfKind::MOE_GLU) {
        if (S.shared_ff > 0) for (Weight* w : {&M.sh_glu, &M.sh_up}) pad_for_tensor_cores(*w);
        std::vector<const void*> up, down, gate;
        for (int e = 0; e < S.experts; e++) { up.push_back(M.e_up[(size_t)e].ptr); down.push_back(M.e_down[(size_t)e].ptr); gate.push_back(M.e_gate[(size_t)e].ptr); }
        auto table = [&](const void**& dst, const std::vector<const void*>& v) {
            dst = dmalloc0<const void*>(v.size());
            NT_CUDA_CHECK(cudaMemcpy(dst, v.data(), sizeof(void*) * v.size(), cudaMemcpyHostToDevice));
        };
        table(M.e_up_tab, up); table(M.e_down_tab, down); table(M.e_gate_tab, gate);
        make_expert_maps(S, M);
    }
    return true;
}

size_t Model::parallel_scratch_width() const {
    size_t m = 1;
    for (const LayerSpec& S : cfg_.layers) m = std::max(m, layer_floats(S, (size_t)cfg_.hidden_size));
    return m + kSlack;
}

void Model::finalize_parallel_decode() {
    const size_t W = (size_t)cfg_.hidden_size;
    par_dec_.slot = up4(W);
    par_dec_.slots = dmalloc0<float>((size_t)(cfg_.n_layers + 1) * par_dec_.slot);
    par_dec_.h = dmalloc0<float>(W);
    for (float*& m : par_dec_.mix) m = dmalloc0<float>(W);
    par_dec_.wide = dmalloc0<float>(parallel_scratch_width());
    size_t seg = 0;
    for (const LayerSpec& S : cfg_.layers) if (S.mixer == MixerKind::WKV) seg = std::max(seg, wkv_rows_scratch_floats(S.heads, S.dim));
    if (seg) { wkv_scratch_ = dmalloc0<float>(seg); owned_.push_back(wkv_scratch_); }
}

void Model::ensure_parallel_buffers(size_t T) {
    for (void* p : {(void*)par_.slots, (void*)par_.h, (void*)par_.wide, par_.hs, par_.mix_s[0], par_.mix_s[1], par_.mix_s[2], par_.mix_s[3], par_.mix_s[4]}) if (p) cudaFree(p);
    par_ = ParRows();
    const size_t W = (size_t)cfg_.hidden_size;
    par_.slot = T * up4(W);
    par_.slots = dmalloc0<float>((size_t)(cfg_.n_layers + 1) * par_.slot);
    par_.h = dmalloc0<float>(T * W);
    par_.wide = dmalloc0<float>(T * parallel_scratch_width());
    if (exact32_) return;
    par_.hs = dmalloc0<uint8_t>(gemm_f16_tc_workspace_bytes((int)T, (int)W));
    bool wkv = false;
    for (const LayerSpec& S : cfg_.layers) wkv = wkv || S.mixer == MixerKind::WKV;
    if (wkv) for (void*& p : par_.mix_s) p = dmalloc0<uint8_t>(gemm_f16_tc_workspace_bytes((int)T, (int)W));
}

bool Model::parallel_split_ok(const Weight& w) const { return pf_.ws && (w.tc_ptr || spec_tc_ok(w)); }

// C [T, w.rows] (+)= A . W^T for prompt rows: tensor cores from the split when the matrix qualifies (short ones through their padded copy),
// else FP32 on CUDA cores from A.
void Model::parallel_gemm(float* C, const float* A, const void* A_split, const Weight& w, int T, bool add, cudaStream_t s) {
    if (A_split && w.tc_ptr) {
        NT_CHECK(!add, "parallel_gemm: a padded matrix stores its product");
        TcOpts o; o.bf16 = true;
        NT_CHECK(gemm_f16_tc_ws(pf_.tmp, A_split, w.tc_ptr, T, w.tc_rows, w.cols, false, s, o), "prefill GEMM (padded) rejected");
        copy_cols(C, pf_.tmp, T, w.rows, w.tc_rows, s);
        return;
    }
    spec_gemm(C, A, A_split, w, T, add ? DENSE_ADD : DENSE_STORE, nullptr, 1.f, s);
}

// ---- one decoded token ----

// The launch between layers: x_i and the inputs of layer i (i == n_layers: hidden_).  Layer 0 reads the embedding, whose launch has
// already put it into slot 1.
static void token_depth(DepthNorm& p, const ModelConfig& cfg, const LayerWeights* done, int i) {
    p.width = cfg.hidden_size; p.groups = cfg.norm_groups; p.eps = cfg.norm_eps;
    p.n = i + 1;
    p.coef = (i > 0 && cfg.depth_average) ? done->depth_w : nullptr;
}

void Model::step_parallel(cudaStream_t s) {
    const ParDec& B = par_dec_;
    const int* pos_dev = step_dev_ + 1;
    embed_bigram_rows(B.slots, B.slots + B.slot, embd_.ptr, embd_.dtype, cfg_.bigram_buckets > 0 ? bigram_.ptr : nullptr, bigram_.dtype, step_dev_, step_dev_ + 2, 1,
                      cfg_.hidden_size, std::max(1, cfg_.bigram_buckets), cfg_.bigram_prev, cfg_.bigram_cur, pos_dev, 0, s);
    for (int i = 0; i <= cfg_.n_layers; i++) {
        DepthNorm p;
        token_depth(p, cfg_, i > 0 ? &layers_[(size_t)i - 1] : nullptr, i);
        p.X = B.slots; p.slot = B.slot;
        if (i == cfg_.n_layers) { p.x_out = hidden_; depth_norm_rows(p, 1, s); break; }
        LayerWeights& L = layers_[(size_t)i];
        p.x_out = i > 0 ? B.slots + (size_t)(i + 1) * B.slot : nullptr;
        p.gain = L.attn_norm; p.h_out = B.h;
        if (cfg_.layers[(size_t)i].mixer == MixerKind::WKV) {
            p.n_mix = 5; p.carried = L.shift_state; p.pos_dev = pos_dev;
            for (int m = 0; m < 5; m++) { p.mu[m] = L.wkv_mu[m]; p.mix_out[m] = B.mix[m]; }
        }
        depth_norm_rows(p, 1, s);
        layer_parallel_token(i, s);
    }
}

void Model::layer_parallel_token(int i, cudaStream_t s) {
    const LayerSpec& S = cfg_.layers[(size_t)i];
    LayerWeights& L = layers_[(size_t)i];
    const ParDec& B = par_dec_;
    const int* pos_dev = step_dev_ + 1;
    const float eps = cfg_.norm_eps;
    float* x = B.slots + (size_t)(i + 1) * B.slot;
    size_t cur = 0;
    auto take = [&](size_t n) { float* p = B.wide + cur; cur += up4(n); return p; };
    const bool moe = S.ff > 0 && S.ff_kind == FfKind::MOE_GLU, mlp = S.ff > 0 && !moe;
    float* act = mlp ? take((size_t)S.ff) : (moe ? take((size_t)S.top * S.ff + S.shared_ff) : nullptr);
    float* logits = moe ? take((size_t)S.experts) : nullptr;
    MultiMat mats[DENSE_MAX_MATS];
    int n = 0;
    float* o = nullptr;
    auto ff_mats = [&]() {
        if (mlp) mats[n++] = multi(L.up, B.h, act, GEMV_ACT_XIELU, L.ff_act);
        if (moe) { MultiMat r; r.W = L.router; r.dtype = DType::F32; r.x = B.h; r.y = logits; r.out = S.experts; r.K = cfg_.hidden_size; mats[n++] = r; }
    };
    if (S.mixer == MixerKind::WKV) {
        const size_t hd = (size_t)S.heads * S.dim;
        float *r = take(hd), *k = take(hd), *v = take(hd), *g = take(hd), *a1 = take((size_t)S.wkv.decay_rank);
        o = take(hd);
        mats[n++] = multi(L.wq, B.mix[0], r); mats[n++] = multi(L.wk, B.mix[1], k); mats[n++] = multi(L.wv, B.mix[2], v); mats[n++] = multi(L.wkv_g, B.mix[3], g);
        mats[n++] = multi(L.wkv_w1, B.mix[4], a1, GEMV_ACT_TANH);
        ff_mats();
        gemv_multi(mats, n, s);
        wkv_token(o, r, k, v, g, a1, L.wkv_w2.ptr, L.wkv_w2.dtype, L.wkv_w0, L.wkv_u, L.wkv_norm, L.wkv_state, eps, S.wkv.decay_rank, S.heads, S.dim, pos_dev, 0, s);
    } else {
        const LatentSpec& A = S.latent;
        const size_t H = (size_t)S.heads;
        float *q = take(H * (size_t)(S.dim + A.rot_dim)), *dkv = take((size_t)A.kv_rank + A.rot_dim), *qa = take(H * (size_t)(A.kv_rank + A.rot_dim)), *ol = take(H * (size_t)A.kv_rank);
        o = take(H * (size_t)S.vdim);
        mats[n++] = multi(L.wq, B.h, q); mats[n++] = multi(L.w_dkv, B.h, dkv);
        ff_mats();
        gemv_multi(mats, n, s);
        latent_prep(nullptr, 0, nullptr, dkv, A.kv_rank, A.rot_dim, L.dkv_norm, eps, kcs_[(size_t)i], cache_dt_, latent_rot(i), 1, pos_dev, 0, s);
        latent_mixer_core(i, 1, pos_dev, 0, q, qa, ol, o, s);
    }
    NT_CHECK(cur <= parallel_scratch_width(), "layer_parallel_token: scratch overrun");
    if (moe) {
        const MoeWeights w = gated_moe(i);
        moe_expert_up_token(act, B.h, nullptr, w, s, logits, moe_sel_, moe_wt_);
    }
    SumTerm t[GEMV_SUM_MAX_TERMS];
    int nt = 0;
    t[nt].W = L.wo.ptr; t[nt].x = o; t[nt++].K = L.wo.cols;
    if (mlp) { t[nt].W = L.down.ptr; t[nt].x = act; t[nt++].K = S.ff; }
    if (moe) {
        bool aligned = true;
        for (const Weight& w : L.e_down) aligned = aligned && (reinterpret_cast<uintptr_t>(w.ptr) & 15) == 0;
        t[nt].table = L.e_down_tab; t[nt].table_aligned = aligned; t[nt].sel = moe_sel_; t[nt].wt = moe_wt_; t[nt].top = S.top; t[nt].x = act; t[nt++].K = S.ff;
        if (S.shared_ff > 0) { t[nt].W = L.sh_down.ptr; t[nt].x = act + (size_t)S.top * S.ff; t[nt++].K = S.shared_ff; }
    }
    gemv_sum(x, t, nt, cfg_.hidden_size, L.wo.dtype, true, s);
}

MoeWeights Model::gated_moe(int i) const {
    const LayerSpec& S = cfg_.layers[(size_t)i];
    const LayerWeights& L = layers_[(size_t)i];
    MoeWeights w;
    w.router = L.router; w.up = L.e_up_tab; w.down = L.e_down_tab; w.gate = L.e_gate_tab; w.dtype = L.e_up[0].dtype;
    w.experts = S.experts; w.top = S.top; w.ff = S.ff; w.width = cfg_.hidden_size;
    w.all = true; w.scale = S.route.scale; w.renorm = S.route.renorm; w.groups = S.route.groups; w.keep = S.route.keep;
    if (S.shared_ff > 0) { w.shared_up = L.sh_up.ptr; w.shared_down = L.sh_down.ptr; w.shared_gatew = L.sh_glu.ptr; w.shared_ff = S.shared_ff; }
    return w;
}

// ---- prompt rows ----

void Model::prefill_parallel(int T, int p0, cudaStream_t s) {
    ParRows& B = par_;
    const size_t W = (size_t)cfg_.hidden_size;
    embed_bigram_rows(B.slots, B.slots + B.slot, embd_.ptr, embd_.dtype, cfg_.bigram_buckets > 0 ? bigram_.ptr : nullptr, bigram_.dtype, pf_.tok, step_dev_, T, (int)W,
                      std::max(1, cfg_.bigram_buckets), cfg_.bigram_prev, cfg_.bigram_cur, nullptr, p0, s);
    // the step's last token is what the next step's first pair looks back at
    NT_CUDA_CHECK(cudaMemcpyAsync(step_dev_, pf_.tok + (T - 1), sizeof(int), cudaMemcpyDeviceToDevice, s));
    for (int i = 0; i <= cfg_.n_layers; i++) {
        DepthNorm p;
        token_depth(p, cfg_, i > 0 ? &layers_[(size_t)i - 1] : nullptr, i);
        p.X = B.slots; p.slot = B.slot;
        if (i == cfg_.n_layers) { p.x_out = pf_.x; depth_norm_rows(p, T, s); break; }
        const LayerSpec& S = cfg_.layers[(size_t)i];
        const LayerWeights& L = layers_[(size_t)i];
        p.x_out = i > 0 ? B.slots + (size_t)(i + 1) * B.slot : nullptr;
        p.gain = L.attn_norm; p.h_out = B.h;
        bool split = S.mixer == MixerKind::ATTN_LATENT && (parallel_split_ok(L.wq) || parallel_split_ok(L.w_dkv));
        if (S.ff > 0 && S.ff_kind == FfKind::MLP) split = split || parallel_split_ok(L.up);
        if (S.shared_ff > 0) split = split || parallel_split_ok(L.sh_glu) || parallel_split_ok(L.sh_up);
        if (split) { p.split = B.hs; p.split_lo = ((size_t)T + 127) / 128 * 128 * W; }
        depth_norm_rows(p, T, s);
        layer_parallel_rows(i, T, p0, s);
    }
}

void Model::layer_parallel_rows(int i, int T, int p0, cudaStream_t s) {
    const LayerSpec& S = cfg_.layers[(size_t)i];
    LayerWeights& L = layers_[(size_t)i];
    const ParRows& B = par_;
    const int W = cfg_.hidden_size;
    const float eps = cfg_.norm_eps;
    float* x = B.slots + (size_t)(i + 1) * B.slot;
    size_t cur = 0;
    auto take = [&](size_t n) { float* p = B.wide + cur; cur += up4(n * (size_t)T); return p; };
    auto hs_of = [&](const Weight& w) { return parallel_split_ok(w) ? B.hs : nullptr; };
    // slot += rows . w^T from F32 rows, split here when the matrix takes the tensor cores
    auto add_product = [&](const float* rows, const Weight& w) {
        const bool tc = parallel_split_ok(w);
        if (tc) split_activations(pf_.ws, rows, T, w.cols, s, true);
        parallel_gemm(x, rows, tc ? pf_.ws : nullptr, w, T, true, s);
    };
    if (S.mixer == MixerKind::WKV) {
        const size_t hd = (size_t)S.heads * S.dim;
        const Weight* w5[5] = {&L.wq, &L.wk, &L.wv, &L.wkv_g, &L.wkv_w1};
        float *r = take(hd), *k = take(hd), *v = take(hd), *g = take(hd), *a = take(hd), *a1 = take((size_t)S.wkv.decay_rank), *ruk = take((size_t)S.heads), *o = take(hd);
        float* y5[5] = {r, k, v, g, a1};
        ShiftMix sm;
        sm.n = 5; sm.split_lo = ((size_t)T + 127) / 128 * 128 * (size_t)W;
        for (int m = 0; m < 5; m++) {
            sm.mu[m] = L.wkv_mu[m];
            if (parallel_split_ok(*w5[m])) sm.split[m] = B.mix_s[m]; else sm.out[m] = take((size_t)W);
        }
        shift_mix_rows(sm, B.h, L.shift_state, T, W, nullptr, p0, s);
        for (int m = 0; m < 5; m++) parallel_gemm(y5[m], sm.out[m], sm.split[m], *w5[m], T, false, s);
        tanh_rows(a1, (size_t)T * S.wkv.decay_rank, s);
        const bool w2_tc = parallel_split_ok(L.wkv_w2);
        if (w2_tc) split_activations(pf_.ws, a1, T, S.wkv.decay_rank, s, true);
        parallel_gemm(a, a1, w2_tc ? pf_.ws : nullptr, L.wkv_w2, T, false, s);
        wkv_prep(a, ruk, r, k, L.wkv_w0, L.wkv_u, T, S.heads, S.dim, s);
        wkv_rows(o, r, k, v, a, ruk, L.wkv_state, T, S.heads, S.dim, nullptr, p0, s, wkv_scratch_);
        const bool o_tc = parallel_split_ok(L.wo);
        wkv_out_norm(o_tc ? nullptr : o, o_tc ? pf_.ws : nullptr, o, g, L.wkv_norm, eps, T, S.heads, S.dim, s);
        parallel_gemm(x, o, o_tc ? pf_.ws : nullptr, L.wo, T, true, s);
    } else {
        const LatentSpec& A = S.latent;
        const size_t H = (size_t)S.heads;
        float *q = take(H * (size_t)(S.dim + A.rot_dim)), *dkv = take((size_t)A.kv_rank + A.rot_dim), *qa = take(H * (size_t)(A.kv_rank + A.rot_dim)), *ol = take(H * (size_t)A.kv_rank),
              *o = take(H * (size_t)S.vdim);
        parallel_gemm(q, B.h, hs_of(L.wq), L.wq, T, false, s);
        parallel_gemm(dkv, B.h, hs_of(L.w_dkv), L.w_dkv, T, false, s);
        latent_prep(nullptr, 0, nullptr, dkv, A.kv_rank, A.rot_dim, L.dkv_norm, eps, kcs_[(size_t)i], cache_dt_, latent_rot(i), T, nullptr, p0, s);
        latent_mixer_core(i, T, nullptr, p0, q, qa, ol, o, s);
        add_product(o, L.wo);
    }
    if (S.ff > 0 && S.ff_kind == FfKind::MLP) {
        const bool tc = parallel_split_ok(L.down);
        if (tc && pf_.ws2 && spec_tc_ok(L.up) && S.ff % 8 == 0) {
            // the activation and the split for the down product in the up GEMM's epilogue: the [T, ff] numbers never reach HBM in FP32
            TcOpts o; o.bf16 = true;
            NT_CHECK(gemm_f16_tc_xielu_ws(pf_.ws2, B.hs, L.up.ptr, L.ff_act, T, S.ff, W, s, o), "prefill GEMM (up) rejected");
            parallel_gemm(x, nullptr, pf_.ws2, L.down, T, true, s);
            NT_CHECK(cur <= parallel_scratch_width() * (size_t)T, "layer_parallel_rows: scratch rows overrun");
            return;
        }
        float* u = take((size_t)S.ff);
        parallel_gemm(u, B.h, hs_of(L.up), L.up, T, false, s);
        xielu_rows(tc ? nullptr : u, tc ? pf_.ws : nullptr, u, L.ff_act, T, S.ff, s);
        parallel_gemm(x, u, tc ? pf_.ws : nullptr, L.down, T, true, s);
    } else if (S.ff > 0) {
        const MoeWeights w = gated_moe(i);
        moe_route(pf_.sel, pf_.wt, nullptr, B.h, w, T, s);
        moe_glu_rows(i, T, B.h, w, x, true, s);
        if (S.shared_ff > 0 && pf_.ws && pf_.ws2 && spec_tc_ok(L.sh_glu) && spec_tc_ok(L.sh_up) && spec_tc_ok(L.sh_down) && S.shared_ff % 128 == 0) {
            TcOpts o; o.bf16 = true;
            NT_CHECK(gemm_f16_tc_swiglu_ws(pf_.ws2, B.hs, L.sh_glu.ptr, L.sh_up.ptr, T, S.shared_ff, W, s, o), "prefill GEMM (shared gate / up) rejected");
            parallel_gemm(x, nullptr, pf_.ws2, L.sh_down, T, true, s);
        } else if (S.shared_ff > 0) {
            float *g = take((size_t)S.shared_ff), *u = take((size_t)S.shared_ff);
            parallel_gemm(g, B.h, hs_of(L.sh_glu), L.sh_glu, T, false, s);
            parallel_gemm(u, B.h, hs_of(L.sh_up), L.sh_up, T, false, s);
            glu_mul(g, g, u, (size_t)T * S.shared_ff, false, s);
            add_product(g, L.sh_down);
        }
    }
    NT_CHECK(cur <= parallel_scratch_width() * (size_t)T, "layer_parallel_rows: scratch rows overrun");
}

}}  // namespace nt::b200
