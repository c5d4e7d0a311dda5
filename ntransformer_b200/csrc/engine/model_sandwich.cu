// model_sandwich.cu — layers of BlockForm::SANDWICH for the resident layer-spec model (engine/model_spec.cu): a norm in front of and behind each
// sublayer, x += n(mixer(n(x, g1)), g1b); x += n(ff(n(x, g2)), g2b).  The mixer is attention with a distance bias, a unit sink, per-head query / key
// norm, a position-dependent query multiplier and one output gate per head (a layer may read an earlier layer's cache rows); latent attention with
// a query latent and an output gate per channel; or the matrix memory (MixerKind::MLSTM).  The feed-forward is W_down relu(W_up h)^2, routed SiLU-gated
// experts with a gated shared one, or absent.
//
// Everything between two sublayers — norm of the output, residual sum, norm of the next input — is one launch (sandwich_norm_rows), so a decoded
// token takes
//   attention layer, 6:  [q, k, v, gate rows]  [head norm, query multiplier, cache write]  [attention]  [merge, gated]  [W_o]  [between]
//   latent layer, 7:     [query latent, key / value latent, gate]  [queries from the normed latent]  [absorbed queries + cache row]  [attention]
//                        [merge + values, gated]  [W_o]  [between]
//   matrix memory, 4:    [q, k, v, gate, input / forget gate rows]  [gates, memory, head norm, output gate]  [W_o]  [between]
//   dense feed-forward, 3:  [relu(W_up .)^2]  [W_down]  [between]      experts, 3:  (router logits come with the launch between mixer and feed-forward)
//                        [choice + experts and shared one up]  [down, weighted]  [between]
// Prompt rows take the tensor-core GEMMs, the tiled attention kernels and the tiled recurrence.  What a sequence carries between steps — cache rows, the
// matrix memory with its normalizer and stabilizer — is written by the step that owns the tokens and read by later steps only from there; the memory
// reads as zeros when a step starts at position 0, so a new request needs no clearing.
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
constexpr int kPadRows = 128;                    // rows of a zero-padded short matrix (Weight::tc_rows)
size_t up4(size_t n) { return (n + 3) & ~(size_t)3; }
size_t padded(size_t n) { return std::max<size_t>(n, kPadRows) + (n < kPadRows ? n : 0); }      // a short product in its padded form and packed
MultiMat multi(const Weight& w, const float* x, float* y, GemvAct act = GEMV_ACT_NONE) {
    MultiMat m;
    m.W = w.ptr; m.dtype = w.dtype; m.row_pitch = w.pitch; m.x = x; m.y = y; m.out = w.rows; m.K = w.cols; m.act = act;
    return m;
}
// floats per row of one layer's intermediates: the decode step's and the prompt pass's layouts both fit (mixer and feed-forward follow each other)
size_t layer_floats(const LayerSpec& S) {
    const size_t H = (size_t)S.heads, G = (size_t)S.kv_heads, D = (size_t)S.dim, V = (size_t)S.vdim;
    size_t mix = 0, ff = 0;
    if (S.mixer == MixerKind::MLSTM) mix = 2 * padded(H * D) + 2 * padded(H * V) + padded(2 * H) + 4 * H + H * V;
    else if (S.mixer == MixerKind::ATTN_LATENT) {
        const size_t r = (size_t)S.latent.kv_rank, R = (size_t)S.latent.rot_dim;
        mix = padded((size_t)S.latent.q_rank) + padded(r + R) + padded(H * V) + padded(H * (D + R)) + H * (r + R) + H * r + H * V;
    } else mix = padded(H * D) + padded(G * D) + padded(G * V) + padded(H) + H * V;
    if (S.ff > 0 && S.ff_kind == FfKind::MLP) ff = padded((size_t)S.ff);
    if (S.ff > 0 && S.ff_kind == FfKind::MOE_GLU) ff = (size_t)S.experts + (size_t)S.top * S.ff + S.shared_ff + 2 * padded((size_t)S.shared_ff);
    return std::max(mix, ff);
}
constexpr size_t kSlack = 64;                    // alignment gaps between the buffers carved from a layer's intermediates
}  // namespace

bool Model::finalize_sandwich_layer(int i) {
    const LayerSpec& S = cfg_.layers[(size_t)i];
    LayerWeights& M = layers_[(size_t)i];
    auto refuse = [&](const char* why) { fprintf(stderr, "model: layer %d: %s\n", i, why); return false; };
    if (S.weights_of >= 0 || cfg_.norm_groups != 1 || cfg_.residual_mult != 1.f) return refuse("shared tensors, grouped norms and residual multipliers are not covered in the sandwich block");
    bool ok = M.attn_norm && M.norm1b && M.wo.ptr && (S.ff == 0 || (M.ffn_norm && M.norm2b));
    std::vector<Weight*> mats = {&M.wo}, pad;
    if (S.mixer == MixerKind::ATTN_WINDOW) {
        if (S.maps != 1 || S.window > 0 || S.chunk > 0 || S.softcap != 0.f || S.conv > 0 || S.qkv_bias || S.talking || S.head_temp || S.sink || S.v_first >= 0 || S.rot.dims > 0 ||
            S.qk_norm != QKNorm::UNIT || S.out_gate == OutGate::PER_CHANNEL)
            return refuse("this attention has no kernels in the sandwich block");
        if (S.dim > 1024 || S.vdim > 512) return refuse("heads wider than 1024 (keys) / 512 (values) are not covered");
        mats.push_back(&M.wq);
        if (S.kv_from < 0) mats.insert(mats.end(), {&M.wk, &M.wv});
    } else if (S.mixer == MixerKind::ATTN_LATENT) {
        if (S.kv_from >= 0 || S.window > 0 || S.out_gate == OutGate::PER_HEAD || S.latent.q_rank <= 0) return refuse("this latent attention has no kernels in the sandwich block");
        if (S.latent.kv_rank > 512) return refuse("latents wider than 512 are not covered");
        ok = ok && M.dq_norm && M.dkv_norm;
        mats.insert(mats.end(), {&M.w_dq, &M.w_uq, &M.w_dkv, &M.w_uk, &M.w_uv});
        pad = {&M.w_dq, &M.w_dkv, &M.w_uq};
    } else if (S.mixer == MixerKind::MLSTM) {
        if (S.dim > MLSTM_MAX_DIM) return refuse("matrix-memory heads wider than 512 are not covered");
        if (S.out_gate != OutGate::PER_CHANNEL || S.kv_heads != S.heads) return refuse("the matrix memory has an output gate per channel and a key head per head");
        ok = ok && M.ml_ib && M.ml_fb && M.ml_norm;
        mats.insert(mats.end(), {&M.wq, &M.wk, &M.wv, &M.ml_i, &M.ml_f});
    } else return refuse("this mixer has no kernels in the sandwich block");
    if (S.mixer != MixerKind::ATTN_LATENT) { pad.push_back(&M.wq); if (S.kv_from < 0) pad.insert(pad.end(), {&M.wk, &M.wv}); }
    if (S.out_gate != OutGate::NONE) { mats.push_back(&M.out_gate); pad.push_back(&M.out_gate); }
    if (S.ff > 0 && S.ff_kind == FfKind::MLP) {
        if (S.act != GluAct::RELU2 || S.ff_bias) return refuse("this feed-forward activation is not covered in the sandwich block");
        mats.insert(mats.end(), {&M.up, &M.down});
        pad.push_back(&M.up);
    } else if (S.ff > 0 && S.ff_kind == FfKind::MOE_GLU) {
        if (!S.route.all || S.act != GluAct::SILU || (S.shared_ff > 0 && !S.shared_glu)) return refuse("this router is not covered in the sandwich block");
        ok = ok && M.router && (int)M.e_up.size() == S.experts && (int)M.e_down.size() == S.experts && (int)M.e_gate.size() == S.experts;
        for (int e = 0; ok && e < S.experts; e++) mats.insert(mats.end(), {&M.e_up[(size_t)e], &M.e_down[(size_t)e], &M.e_gate[(size_t)e]});
        if (S.shared_ff > 0) { mats.insert(mats.end(), {&M.sh_glu, &M.sh_up, &M.sh_down}); pad.insert(pad.end(), {&M.sh_glu, &M.sh_up}); }
    } else if (S.ff > 0) return refuse("this feed-forward is not covered in the sandwich block");
    for (const Weight* w : mats) ok = ok && w->ptr;
    if (!ok) return refuse("tensors are missing");
    for (const Weight* w : mats)
        if (w->dtype != mats[0]->dtype || w->pitch != dtype_row_size(w->dtype, (size_t)w->cols)) return refuse("its matrices must have one dtype and packed rows");
    for (Weight* w : pad) pad_for_tensor_cores(*w);
    auto table = [&](const std::vector<float>& v) {
        float* d = dmalloc0<float>(v.size());
        NT_CUDA_CHECK(cudaMemcpy(d, v.data(), sizeof(float) * v.size(), cudaMemcpyHostToDevice));
        owned_.push_back(d);
        return d;
    };
    if (S.distance_bias) {
        std::vector<float> v;
        for (int h = 0; h < S.heads; h++) v.push_back((float)std::exp2(-8.0 * (h + 1) / S.heads));
        M.slopes = table(v);
    }
    if (S.unit_sink) M.zero_sink = table(std::vector<float>((size_t)S.heads, 0.f));
    if (S.mixer == MixerKind::ATTN_LATENT && S.rot.dims > 0 && S.rot.factor > 0.0) {
        const RotarySpec& R = S.rot;
        std::vector<double> f((size_t)R.dims / 2);
        M.rot_mag = rotary_table(f.data(), R.dims, R.base, R.factor, R.original, R.fast, R.slow);
        M.rot_freq64 = dmalloc0<double>(f.size());
        NT_CUDA_CHECK(cudaMemcpy(M.rot_freq64, f.data(), sizeof(double) * f.size(), cudaMemcpyHostToDevice));
    }
    if (S.mixer == MixerKind::MLSTM) {
        M.ml_state = dmalloc0<float>((size_t)S.heads * (S.vdim + 1) * S.dim);
        M.ml_m = dmalloc0<float>((size_t)S.heads);
        // prompt rows: the two short gate matrices as one product, forget gate rows behind the input gate's
        const size_t bytes = (size_t)S.heads * M.ml_i.pitch;
        Weight w = M.ml_i;
        w.rows = 2 * S.heads;
        if (w.dtype == DType::BF16 && w.rows < kPadRows) {
            uint8_t* p = dmalloc0<uint8_t>(2 * bytes);
            NT_CUDA_CHECK(cudaMemcpy(p, M.ml_i.ptr, bytes, cudaMemcpyDeviceToDevice));
            NT_CUDA_CHECK(cudaMemcpy(p + bytes, M.ml_f.ptr, bytes, cudaMemcpyDeviceToDevice));
            owned_.push_back(p);
            w.ptr = p;
            pad_for_tensor_cores(w);
            if (w.tc_ptr) M.ml_if = w;
        }
    }
    if (S.ff > 0 && S.ff_kind == FfKind::MOE_GLU) {
        std::vector<const void*> up, down, gate;
        for (int e = 0; e < S.experts; e++) { up.push_back(M.e_up[(size_t)e].ptr); down.push_back(M.e_down[(size_t)e].ptr); gate.push_back(M.e_gate[(size_t)e].ptr); }
        auto ptr_table = [&](const void**& dst, const std::vector<const void*>& v) {
            dst = dmalloc0<const void*>(v.size());
            NT_CUDA_CHECK(cudaMemcpy(dst, v.data(), sizeof(void*) * v.size(), cudaMemcpyHostToDevice));
        };
        ptr_table(M.e_up_tab, up); ptr_table(M.e_down_tab, down); ptr_table(M.e_gate_tab, gate);
        make_expert_maps(S, M);
    }
    return true;
}

size_t Model::sandwich_scratch_width() const {
    size_t m = 1;
    for (const LayerSpec& S : cfg_.layers) m = std::max(m, layer_floats(S));
    return m + kSlack;
}

void Model::finalize_sandwich_decode() {
    dec_.y = dmalloc0<float>((size_t)cfg_.hidden_size);
    for (int t = 0; t < 2; t++) dec_.t[t] = dmalloc0<float>((size_t)cfg_.hidden_size);
    int experts = 1;
    for (const LayerSpec& S : cfg_.layers) if (S.ff_kind == FfKind::MOE_GLU) experts = std::max(experts, S.experts);
    moe_logits_ = dmalloc0<float>((size_t)experts);
    owned_.push_back(moe_logits_);
    dec_.wide = dmalloc0<float>(sandwich_scratch_width());
    size_t seg = 0;
    for (const LayerSpec& S : cfg_.layers) if (S.mixer == MixerKind::MLSTM) seg = std::max(seg, mlstm_rows_scratch_floats(S.heads, S.dim, S.vdim));
    if (seg) { ml_scratch_ = dmalloc0<float>(seg); owned_.push_back(ml_scratch_); }
}

static HeadPrep head_prep_of(const LayerSpec& S, float eps) {
    HeadPrep p;
    p.heads = S.heads; p.kv_heads = S.kv_heads; p.dim = S.dim; p.vdim = S.vdim; p.eps = eps; p.unit_norm = S.qk_norm == QKNorm::UNIT ? 1 : 0;
    p.temp_coef = S.q_temp.coef; p.temp_every = S.q_temp.every;
    return p;
}
static WindowAttn biased_attn_of(const LayerSpec& S, const LayerWeights& L) {
    WindowAttn a;
    a.heads = S.heads; a.kv_heads = S.kv_heads; a.dim = S.dim; a.vdim = S.vdim; a.scale = S.scale; a.sink = L.zero_sink; a.slope = L.slopes;
    return a;
}

// ---- one decoded token ----

void Model::step_sandwich(cudaStream_t s) {
    const int W = cfg_.hidden_size;
    const float eps = cfg_.norm_eps;
    // a launch that also routes writes the residual into the other of two rows; start so that the last result lands in hidden_
    float *x = hidden_, *other = dec_.t[1], *h = dec_.t[0], *y = dec_.y;
    int routed_layers = 0;
    for (const LayerSpec& S : cfg_.layers) routed_layers += S.ff > 0 && S.ff_kind == FfKind::MOE_GLU;
    if (routed_layers & 1) std::swap(x, other);
    embed_rows(x, embd_.ptr, embd_.dtype, step_dev_, 1, W, s);
    sandwich_norm_rows(x, nullptr, nullptr, layers_[0].attn_norm, h, nullptr, 1, W, eps, s);
    for (int i = 0; i < cfg_.n_layers; i++) {
        const LayerWeights& L = layers_[(size_t)i];
        const float* next = i + 1 < cfg_.n_layers ? layers_[(size_t)i + 1].attn_norm : nullptr;       // the head normalises the last result itself
        const bool ff = cfg_.layers[(size_t)i].ff > 0;
        sandwich_mixer_token(i, y, s);
        const bool routed = ff && cfg_.layers[(size_t)i].ff_kind == FfKind::MOE_GLU;
        const bool with_logits = routed && sandwich_norm_router(other, x, y, L.norm1b, L.ffn_norm, h, L.router, moe_logits_, cfg_.layers[(size_t)i].experts, W, eps, s);
        if (with_logits) std::swap(x, other);
        else sandwich_norm_rows(x, y, L.norm1b, ff ? L.ffn_norm : next, h, nullptr, 1, W, eps, s);
        if (!ff) continue;
        sandwich_ff_token(i, y, with_logits, s);
        sandwich_norm_rows(x, y, L.norm2b, next, h, nullptr, 1, W, eps, s);
    }
    if (x != hidden_) copy(hidden_, x, W, s);
}

// y = mixer(h), h = dec_.t[0]
void Model::sandwich_mixer_token(int i, float* y, cudaStream_t s) {
    const LayerSpec& S = cfg_.layers[(size_t)i];
    LayerWeights& L = layers_[(size_t)i];
    const float* h = dec_.t[0];
    const int* pos_dev = step_dev_ + 1;
    const float eps = cfg_.norm_eps;
    const size_t H = (size_t)S.heads, G = (size_t)S.kv_heads, D = (size_t)S.dim, V = (size_t)S.vdim;
    size_t cur = 0;
    auto take = [&](size_t n) { float* p = dec_.wide + cur; cur += up4(n); return p; };
    MultiMat mats[DENSE_MAX_MATS];
    int n = 0;
    float *o = take(H * V), *g = S.out_gate != OutGate::NONE ? take((size_t)L.out_gate.rows) : nullptr;
    if (S.mixer == MixerKind::ATTN_WINDOW) {
        float *q = take(H * D), *k = nullptr, *v = nullptr;
        mats[n++] = multi(L.wq, h, q);
        if (S.kv_from < 0) { k = take(G * D); v = take(G * V); mats[n++] = multi(L.wk, h, k); mats[n++] = multi(L.wv, h, v); }
        if (g) mats[n++] = multi(L.out_gate, h, g);
        gemv_multi(mats, n, s);
        void *kc = kcs_[(size_t)i], *vc = vcs_[(size_t)i];
        head_prep(q, k, v, head_prep_of(S, eps), kc, vc, cache_dt_, 1, pos_dev, 0, s);
        WindowAttn a = biased_attn_of(S, L);
        a.head_gate = g; a.gate_stride = S.heads; a.scratch = lat_part_;
        attention_window(o, q, kc, vc, cache_dt_, 1, pos_dev, 0, cfg_.max_seq_len, a, s);
    } else if (S.mixer == MixerKind::ATTN_LATENT) {
        const LatentSpec& A = S.latent;
        const size_t r = (size_t)A.kv_rank, R = (size_t)A.rot_dim;
        float *cq = take((size_t)A.q_rank), *dkv = take(r + R), *q = take(H * (D + R)), *qa = take(H * (r + R)), *ol = take(H * r);
        mats[n++] = multi(L.w_dq, h, cq); mats[n++] = multi(L.w_dkv, h, dkv);
        if (g) mats[n++] = multi(L.out_gate, h, g);
        gemv_multi(mats, n, s);
        mats[0] = multi(L.w_uq, cq, q);
        mats[0].norm_w = L.dq_norm; mats[0].eps = eps;
        gemv_multi(mats, 1, s);
        LatentRow row;
        row.dkv = dkv; row.gain = L.dkv_norm; row.eps = eps; row.cache = kcs_[(size_t)i]; row.cache_dt = cache_dt_;
        latent_mixer_core(i, 1, pos_dev, 0, q, qa, ol, o, s, g, &row);
    } else {
        float *q = take(H * D), *k = take(H * D), *v = take(H * V), *zi = take(H), *zf = take(H);
        mats[n++] = multi(L.wq, h, q); mats[n++] = multi(L.wk, h, k); mats[n++] = multi(L.wv, h, v); mats[n++] = multi(L.out_gate, h, g);
        mats[n++] = multi(L.ml_i, h, zi); mats[n++] = multi(L.ml_f, h, zf);
        gemv_multi(mats, n, s);
        mlstm_token(o, q, k, v, g, zi, zf, L.ml_ib, L.ml_fb, L.ml_norm, L.ml_state, L.ml_m, S.mlstm.gate_cap, 1.0f / std::sqrt((float)S.dim), eps, S.heads, S.dim, S.vdim, pos_dev, 0, s);
    }
    NT_CHECK(cur <= sandwich_scratch_width(), "sandwich_mixer_token: scratch overrun");
    SumTerm t;
    t.W = L.wo.ptr; t.x = o; t.K = L.wo.cols;
    gemv_sum(y, &t, 1, cfg_.hidden_size, L.wo.dtype, false, s);
}

// y = ff(h), h = dec_.t[0]; with_logits: the router's logits are already in moe_logits_
void Model::sandwich_ff_token(int i, float* y, bool with_logits, cudaStream_t s) {
    const LayerSpec& S = cfg_.layers[(size_t)i];
    const LayerWeights& L = layers_[(size_t)i];
    const float* h = dec_.t[0];
    size_t cur = 0;
    auto take = [&](size_t n) { float* p = dec_.wide + cur; cur += up4(n); return p; };
    SumTerm t[2];
    int nt = 0;
    if (S.ff_kind == FfKind::MLP) {
        float* a = take((size_t)S.ff);
        const MultiMat m = multi(L.up, h, a, GEMV_ACT_RELU2);
        gemv_multi(&m, 1, s);
        t[nt].W = L.down.ptr; t[nt].x = a; t[nt++].K = S.ff;
    } else {
        float* act = take((size_t)S.top * S.ff + S.shared_ff);
        if (!with_logits) {
            MultiMat m;
            m.W = L.router; m.dtype = DType::F32; m.x = h; m.y = moe_logits_; m.out = S.experts; m.K = cfg_.hidden_size;
            gemv_multi(&m, 1, s);
        }
        const MoeWeights w = gated_moe(i);
        moe_expert_up_token(act, h, nullptr, w, s, moe_logits_, moe_sel_, moe_wt_);
        bool aligned = true;
        for (const Weight& d : L.e_down) aligned = aligned && (reinterpret_cast<uintptr_t>(d.ptr) & 15) == 0;
        t[nt].table = L.e_down_tab; t[nt].table_aligned = aligned; t[nt].sel = moe_sel_; t[nt].wt = moe_wt_; t[nt].top = S.top; t[nt].x = act; t[nt++].K = S.ff;
        if (S.shared_ff > 0) { t[nt].W = L.sh_down.ptr; t[nt].x = act + (size_t)S.top * S.ff; t[nt++].K = S.shared_ff; }
    }
    NT_CHECK(cur <= sandwich_scratch_width(), "sandwich_ff_token: scratch overrun");
    gemv_sum(y, t, nt, cfg_.hidden_size, L.wo.dtype, false, s);
}

// ---- prompt rows ----

void Model::prefill_sandwich(int T, int p0, cudaStream_t s) {
    const int W = cfg_.hidden_size;
    const float eps = cfg_.norm_eps;
    float *x = pf_.x, *y = pf_.tmp;
    embed_rows(x, embd_.ptr, embd_.dtype, pf_.tok, T, W, s);
    // h = n(x, gain) in the forms the sublayer reads: F32 rows (CUDA-core products, the router, the experts' gather), the BF16 split, or both
    auto between = [&](const float* y_in, const float* gain_y, int layer, bool ff) {
        if (layer >= cfg_.n_layers) { sandwich_norm_rows(x, y_in, gain_y, nullptr, nullptr, nullptr, T, W, eps, s); return; }
        const LayerSpec& S = cfg_.layers[(size_t)layer];
        const LayerWeights& L = layers_[(size_t)layer];
        bool f32 = false, split = false;
        auto reads = [&](const Weight& w) { if (!w.ptr) return; if (rows_take_tc(w)) split = true; else f32 = true; };
        if (!ff) {
            if (S.mixer == MixerKind::ATTN_LATENT) { reads(L.w_dq); reads(L.w_dkv); }
            else { reads(L.wq); if (S.kv_from < 0) { reads(L.wk); reads(L.wv); } }
            if (S.mixer == MixerKind::MLSTM) reads(L.ml_if.ptr ? L.ml_if : L.ml_i);
            reads(L.out_gate);
        } else if (S.ff_kind == FfKind::MLP) reads(L.up);
        else { f32 = true; reads(L.sh_glu); reads(L.sh_up); }
        sandwich_norm_rows(x, y_in, gain_y, ff ? L.ffn_norm : L.attn_norm, f32 ? pf_.h : nullptr, split ? pf_.hws : nullptr, T, W, eps, s);
    };
    between(nullptr, nullptr, 0, false);
    for (int i = 0; i < cfg_.n_layers; i++) {
        const LayerWeights& L = layers_[(size_t)i];
        sandwich_mixer_rows(i, T, p0, y, s);
        if (cfg_.layers[(size_t)i].ff == 0) { between(y, L.norm1b, i + 1, false); continue; }
        between(y, L.norm1b, i, true);
        sandwich_ff_rows(i, T, y, s);
        between(y, L.norm2b, i + 1, false);
    }
}

// y = mixer(h), h in pf_.h / pf_.hws
void Model::sandwich_mixer_rows(int i, int T, int p0, float* y, cudaStream_t s) {
    const LayerSpec& S = cfg_.layers[(size_t)i];
    LayerWeights& L = layers_[(size_t)i];
    const float eps = cfg_.norm_eps;
    const size_t H = (size_t)S.heads, V = (size_t)S.vdim;
    size_t cur = 0;
    auto take = [&](size_t n) { float* p = pf_.wide + cur; cur += up4(n * (size_t)T); return p; };
    // rows . w^T; a short matrix goes through its padded copy, whose product has rows of ld = Weight::tc_rows numbers
    auto product = [&](const Weight& w, const float* A, const void* A_split, int& ld) {
        ld = w.rows;
        if (A_split && w.tc_ptr) {
            ld = w.tc_rows;
            float* C = take((size_t)w.tc_rows);
            TcOpts o; o.bf16 = true;
            NT_CHECK(gemm_f16_tc_ws(C, A_split, w.tc_ptr, T, w.tc_rows, w.cols, false, s, o), "prefill GEMM (padded) rejected");
            return C;
        }
        float* C = take((size_t)w.rows);
        spec_gemm(C, A, A_split, w, T, DENSE_STORE, nullptr, 1.f, s);
        return C;
    };
    auto packed = [&](const Weight& w, const float* A, const void* A_split) {
        int ld = 0;
        float* C = product(w, A, A_split, ld);
        if (ld == w.rows) return C;
        float* P = take((size_t)w.rows);
        copy_cols(P, C, T, w.rows, ld, s);
        return P;
    };
    // the products that read h: those of 256 rows or more are collected and run as one launch, the others at once
    float* many_C[TC_MULTI_MAX];
    const Weight* many[TC_MULTI_MAX];
    int n_many = 0;
    auto of_h = [&](const Weight& w, int* ld = nullptr) {
        if (rows_take_tc(w) && !w.tc_ptr && w.rows >= 256 && n_many < TC_MULTI_MAX) {
            many[n_many] = &w;
            if (ld) *ld = w.rows;
            return many_C[n_many++] = take((size_t)w.rows);
        }
        const void* split = rows_take_tc(w) ? pf_.hws : nullptr;
        return ld ? product(w, pf_.h, split, *ld) : packed(w, pf_.h, split);
    };
    auto run_many = [&]() {
        const void* W[TC_MULTI_MAX];
        int N[TC_MULTI_MAX];
        for (int x = 0; x < n_many; x++) { W[x] = many[x]->ptr; N[x] = many[x]->rows; }
        TcOpts opt; opt.bf16 = true;
        if (n_many == 1) NT_CHECK(gemm_f16_tc_ws(many_C[0], pf_.hws, W[0], T, N[0], cfg_.hidden_size, false, s, opt), "prefill GEMM rejected");
        else if (n_many > 1) NT_CHECK(gemm_f16_tc_multi_ws(many_C, pf_.hws, W, N, n_many, T, cfg_.hidden_size, s, opt), "prefill GEMM (several matrices) rejected");
    };
    const bool o_tc = rows_take_tc(L.wo);
    float* o = take(H * V);
    if (S.mixer == MixerKind::MLSTM) {
        float *q = of_h(L.wq), *k = of_h(L.wk), *v = of_h(L.wv), *g = of_h(L.out_gate);
        run_many();
        int ld = 0;
        const float *zi = nullptr, *zf = nullptr;
        if (L.ml_if.ptr && rows_take_tc(L.ml_if)) { zi = product(L.ml_if, nullptr, pf_.hws, ld); zf = zi + H; }
        else { zi = product(L.ml_i, pf_.h, nullptr, ld); zf = product(L.ml_f, pf_.h, nullptr, ld); }
        float *a = take(H), *b = take(H), *em = take(H), *den = take(H);
        mlstm_gates(a, b, em, zi, zf, ld, L.ml_ib, L.ml_fb, S.mlstm.gate_cap, L.ml_m, T, S.heads, nullptr, p0, s);
        mlstm_rows(o, den, q, k, v, a, b, L.ml_state, 1.0f / std::sqrt((float)S.dim), T, S.heads, S.dim, S.vdim, nullptr, p0, s, ml_scratch_);
        mlstm_out_norm(o_tc ? nullptr : o, o_tc ? pf_.ws : nullptr, o, den, em, g, L.ml_norm, eps, T, S.heads, S.vdim, s);
    } else {
        const float* g = nullptr;
        int g_ld = 0;
        if (S.out_gate != OutGate::NONE) g = of_h(L.out_gate, &g_ld);
        if (S.mixer == MixerKind::ATTN_WINDOW) {
            float *q = of_h(L.wq), *k = nullptr, *v = nullptr;
            if (S.kv_from < 0) { k = of_h(L.wk); v = of_h(L.wv); }
            run_many();
            void *kc = kcs_[(size_t)i], *vc = vcs_[(size_t)i];
            head_prep(q, k, v, head_prep_of(S, eps), kc, vc, cache_dt_, T, nullptr, p0, s);
            attention_window(o, q, kc, vc, cache_dt_, T, nullptr, p0, cfg_.max_seq_len, biased_attn_of(S, L), s);
        } else {
            const LatentSpec& A = S.latent;
            float *cq = of_h(L.w_dq), *dkv = of_h(L.w_dkv);
            run_many();
            latent_prep(cq, A.q_rank, L.dq_norm, dkv, A.kv_rank, A.rot_dim, L.dkv_norm, eps, kcs_[(size_t)i], cache_dt_, latent_rot(i), T, nullptr, p0, s);
            const bool uq_tc = rows_take_tc(L.w_uq);
            if (uq_tc) split_activations(pf_.ws, cq, T, A.q_rank, s, true);
            float *q = packed(L.w_uq, cq, uq_tc ? pf_.ws : nullptr), *qa = take(H * (size_t)(A.kv_rank + A.rot_dim)), *ol = take(H * (size_t)A.kv_rank);
            latent_mixer_core(i, T, nullptr, p0, q, qa, ol, o, s);
        }
        if (g) sigmoid_gate_rows(o_tc ? nullptr : o, o_tc ? pf_.ws : nullptr, o, g, g_ld, S.out_gate == OutGate::PER_HEAD ? S.vdim : 1, T, (int)(H * V), s);
        else if (o_tc) split_activations(pf_.ws, o, T, (int)(H * V), s, true);
    }
    NT_CHECK(cur <= sandwich_scratch_width() * (size_t)T, "sandwich_mixer_rows: scratch rows overrun");
    spec_gemm(y, o, o_tc ? pf_.ws : nullptr, L.wo, T, DENSE_STORE, nullptr, 1.f, s);
}

// y = ff(h), h in pf_.h / pf_.hws
void Model::sandwich_ff_rows(int i, int T, float* y, cudaStream_t s) {
    const LayerSpec& S = cfg_.layers[(size_t)i];
    const LayerWeights& L = layers_[(size_t)i];
    const int W = cfg_.hidden_size;
    size_t cur = 0;
    auto take = [&](size_t n) { float* p = pf_.wide + cur; cur += up4(n * (size_t)T); return p; };
    auto packed = [&](const Weight& w) {
        float* C = take((size_t)w.rows);
        if (w.tc_ptr && rows_take_tc(w)) {
            float* P = take((size_t)w.tc_rows);
            TcOpts o; o.bf16 = true;
            NT_CHECK(gemm_f16_tc_ws(P, pf_.hws, w.tc_ptr, T, w.tc_rows, w.cols, false, s, o), "prefill GEMM (padded) rejected");
            copy_cols(C, P, T, w.rows, w.tc_rows, s);
        } else spec_gemm(C, pf_.h, rows_take_tc(w) ? pf_.hws : nullptr, w, T, DENSE_STORE, nullptr, 1.f, s);
        return C;
    };
    if (S.ff_kind == FfKind::MLP) {
        const bool down_tc = rows_take_tc(L.down);
        if (down_tc && pf_.ws2 && spec_tc_ok(L.up) && S.ff % 8 == 0) {
            // the activation and the split for the down product in the up GEMM's epilogue: the [T, ff] numbers never reach HBM in FP32
            TcOpts o; o.bf16 = true;
            NT_CHECK(gemm_f16_tc_relu2_ws(pf_.ws2, pf_.hws, L.up.ptr, T, S.ff, W, s, o), "prefill GEMM (up) rejected");
            spec_gemm(y, nullptr, pf_.ws2, L.down, T, DENSE_STORE, nullptr, 1.f, s);
            return;
        }
        float* u = packed(L.up);
        relu2_rows(down_tc ? nullptr : u, down_tc ? pf_.ws : nullptr, u, T, S.ff, s);
        spec_gemm(y, u, down_tc ? pf_.ws : nullptr, L.down, T, DENSE_STORE, nullptr, 1.f, s);
    } else {
        const MoeWeights w = gated_moe(i);
        moe_route(pf_.sel, pf_.wt, nullptr, pf_.h, w, T, s);
        moe_glu_rows(i, T, pf_.h, w, y, false, s);
        if (S.shared_ff > 0 && pf_.ws2 && spec_tc_ok(L.sh_glu) && spec_tc_ok(L.sh_up) && spec_tc_ok(L.sh_down) && S.shared_ff % 128 == 0) {
            TcOpts o; o.bf16 = true;
            NT_CHECK(gemm_f16_tc_swiglu_ws(pf_.ws2, pf_.hws, L.sh_glu.ptr, L.sh_up.ptr, T, S.shared_ff, W, s, o), "prefill GEMM (shared gate / up) rejected");
            spec_gemm(y, nullptr, pf_.ws2, L.sh_down, T, DENSE_ADD, nullptr, 1.f, s);
        } else if (S.shared_ff > 0) {
            float *g = packed(L.sh_glu), *u = packed(L.sh_up);
            glu_mul(g, g, u, (size_t)T * S.shared_ff, false, s);
            const bool down_tc = rows_take_tc(L.sh_down);
            if (down_tc) split_activations(pf_.ws, g, T, S.shared_ff, s, true);
            spec_gemm(y, g, down_tc ? pf_.ws : nullptr, L.sh_down, T, DENSE_ADD, nullptr, 1.f, s);
        }
    }
    NT_CHECK(cur <= sandwich_scratch_width() * (size_t)T, "sandwich_ff_rows: scratch rows overrun");
}

}}  // namespace nt::b200
