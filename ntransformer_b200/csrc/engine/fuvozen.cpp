// fuvozen.cpp — the Fuvozen family: a decoder with one norm per layer whose mixer and feed-forward both read it and join the residual
// together (BlockForm::PARALLEL), and whose layer inputs are learned averages over the depth (ModelConfig::depth_average: x <- sum_j
// dwa[j] X_j over the embedding and every layer's result so far).  Norms work on groups of channels (ModelConfig::norm_groups).  A second
// embedding over hashed token pairs joins the first (ModelConfig::bigram_*).  A layer's mixer, in whatever order the configuration lists
// them, is either
//   "latent_attention": low-rank attention with queries straight from h (MixerKind::ATTN_LATENT, LatentSpec::q_rank == 0), interleaved
//                       rotary pairs on the rotated part, softmax over a sliding window (LayerSpec::window); or
//   "wkv":              the WKV time mixer (MixerKind::WKV, WkvSpec).
// The feed-forward is W_down xielu(W_up h) with two learned numbers (FfKind::MLP, GluAct::XIELU), a mixture of SiLU-gated experts
// weighted by the softmax over all of them (FfKind::MOE_GLU, RouteSpec::all) with an optional gated shared expert, or absent
// ("mlp": null).  The head is the embedding table.  Every size and constant that varies between models of the family is read from
// config.json; the rank of the WKV decay is the row count of its first matrix.
#include "model_registry.h"
#include <algorithm>

namespace nt { namespace b200 {

namespace {

bool need_int(const Json& o, const char* key, int& out, std::string& err, const std::string& where) {
    const Json& v = o.at(key);
    if (!v.is_number()) { err = where + ": \"" + key + "\" is missing or not a number"; return false; }
    out = (int)v.int_or(0);
    return true;
}
bool need_float(const Json& o, const char* key, float& out, std::string& err, const std::string& where) {
    const Json& v = o.at(key);
    if (!v.is_number()) { err = where + ": \"" + key + "\" is missing or not a number"; return false; }
    out = (float)v.number_or(0.0);
    return true;
}

bool latent_from_json(const Json& m, LayerSpec& L, std::string& err, const std::string& where) {
    L.mixer = MixerKind::ATTN_LATENT;
    L.kv_heads = 1;
    if (!need_int(m, "heads", L.heads, err, where) || !need_int(m, "dim", L.dim, err, where) || !need_int(m, "vdim", L.vdim, err, where) ||
        !need_int(m, "rot_dim", L.latent.rot_dim, err, where) || !need_int(m, "kv_rank", L.latent.kv_rank, err, where) || !need_float(m, "scale", L.scale, err, where))
        return false;
    if (L.heads <= 0 || L.dim < 0 || L.vdim <= 0 || L.latent.rot_dim < 0 || L.dim + L.latent.rot_dim <= 0 || L.latent.kv_rank <= 0) { err = where + ": invalid mixer sizes"; return false; }
    L.rot.interleaved = true;                  // channel 2i pairs with channel 2i + 1
    if (m.at("rot").is_object()) {
        const Json& r = m.at("rot");
        if (!need_int(r, "dims", L.rot.dims, err, where + ".rot")) return false;
        if (!r.at("base").is_number()) { err = where + ".rot: \"base\" is missing or not a number"; return false; }
        L.rot.base = r.at("base").number_or(0.0);
        if (L.rot.dims < 0 || L.rot.dims > L.latent.rot_dim || (L.rot.dims & 1) || L.rot.base <= 0.0) { err = where + ": rot.dims must be even and at most rot_dim"; return false; }
    }
    if (m.at("mask").is_object()) {
        if (!need_int(m.at("mask"), "size", L.window, err, where + ".mask")) return false;
        if (L.window <= 0) { err = where + ": mask.size must be positive"; return false; }
    }
    return true;
}

bool wkv_from_json(const Json& m, LayerSpec& L, std::string& err, const std::string& where) {
    L.mixer = MixerKind::WKV;
    if (!need_int(m, "heads", L.heads, err, where) || !need_int(m, "dim", L.dim, err, where)) return false;
    if (L.heads <= 0 || L.dim <= 0) { err = where + ": invalid mixer sizes"; return false; }
    if (m.has("decay_rank") && !need_int(m, "decay_rank", L.wkv.decay_rank, err, where)) return false;      // else the rows of its first matrix
    if (L.wkv.decay_rank < 0) { err = where + ": invalid rank"; return false; }
    L.kv_heads = L.heads; L.vdim = L.dim;
    return true;
}

bool ff_from_json(const Json& mlp, LayerSpec& L, std::string& err, const std::string& where) {
    const std::string kind = mlp.at("kind").string_or("");
    if (kind == "dense") {
        L.ff_kind = FfKind::MLP; L.act = GluAct::XIELU;
        if (!need_int(mlp, "ff", L.ff, err, where)) return false;
        if (L.ff <= 0) { err = where + ": invalid ff"; return false; }
        return true;
    }
    if (kind != "moe") { err = where + ": feed-forward kind \"" + kind + "\" is not part of this family"; return false; }
    L.ff_kind = FfKind::MOE_GLU; L.act = GluAct::SILU;
    L.route.all = true;
    const Json& r = mlp.at("router");
    if (!need_int(mlp.at("expert"), "ff", L.ff, err, where + ".expert") || !need_int(r, "experts", L.experts, err, where + ".router") ||
        !need_int(r, "top", L.top, err, where + ".router") || !need_float(r, "scale", L.route.scale, err, where + ".router")) return false;
    if (L.ff <= 0 || L.experts <= 0 || L.top <= 0 || L.top > L.experts || L.experts > 256) { err = where + ": invalid expert sizes (1 <= top <= experts <= 256)"; return false; }
    if (mlp.at("shared").is_object()) {
        L.shared_glu = true;
        if (!need_int(mlp.at("shared"), "ff", L.shared_ff, err, where + ".shared")) return false;
        if (L.shared_ff <= 0) { err = where + ": invalid shared ff"; return false; }
    }
    return true;
}

bool config_from_json(const Json& root, ModelConfig& cfg, std::string& err) {
    if (!need_int(root, "vocab", cfg.vocab_size, err, "config") || !need_int(root, "width", cfg.hidden_size, err, "config")) return false;
    if (!need_float(root.at("norm"), "eps", cfg.norm_eps, err, "config.norm") || !need_int(root.at("norm"), "groups", cfg.norm_groups, err, "config.norm")) return false;
    if (cfg.vocab_size <= 0 || cfg.hidden_size <= 0) { err = "config: invalid vocab / width"; return false; }
    if (cfg.norm_groups <= 0 || cfg.norm_groups > 256 || cfg.hidden_size % cfg.norm_groups) { err = "config.norm: groups must divide the width (1 <= groups <= 256)"; return false; }
    const Json& bg = root.at("embedding").at("bigram");
    if (bg.is_object()) {
        if (!need_int(bg, "buckets", cfg.bigram_buckets, err, "config.embedding.bigram")) return false;
        if (!bg.at("mul_prev").is_number() || !bg.at("mul_cur").is_number()) { err = "config.embedding.bigram: \"mul_prev\" / \"mul_cur\" are missing"; return false; }
        cfg.bigram_prev = bg.at("mul_prev").int_or(0); cfg.bigram_cur = bg.at("mul_cur").int_or(0);
        if (cfg.bigram_buckets <= 0) { err = "config.embedding.bigram: invalid buckets"; return false; }
        // the row only depends on the factors' residues, and residues keep the products in 64 bits
        cfg.bigram_prev %= cfg.bigram_buckets; cfg.bigram_cur %= cfg.bigram_buckets;
    }
    cfg.depth_average = true;
    cfg.tied_head = true;
    const Json& layers = root.at("layers");
    if (!layers.is_array() || layers.arr.empty()) { err = "config: \"layers\" must be a non-empty list"; return false; }
    cfg.n_layers = (int)layers.arr.size();
    cfg.model_name = "fuvozen";
    cfg.bos_token_id = -1; cfg.eos_token_id = -1;
    for (size_t i = 0; i < layers.arr.size(); i++) {
        const Json& e = layers.arr[i];
        const std::string where = "config.layers[" + std::to_string(i) + "]";
        LayerSpec L;
        L.form = BlockForm::PARALLEL;
        const std::string type = e.at("type").string_or("");
        const Json& m = e.at("mixer");
        if (!m.is_object()) { err = where + ": \"mixer\" is missing"; return false; }
        if (type == "latent_attention") { if (!latent_from_json(m, L, err, where)) return false; }
        else if (type == "wkv") { if (!wkv_from_json(m, L, err, where)) return false; }
        else { err = where + ": mixer type \"" + type + "\" is not part of this family"; return false; }
        if (!e.at("mlp").is_null() && !ff_from_json(e.at("mlp"), L, err, where + ".mlp")) return false;
        cfg.layers.push_back(L);
    }
    cfg.n_heads = cfg.n_kv_heads = cfg.head_dim = cfg.intermediate_size = 0;
    for (const LayerSpec& L : cfg.layers) {
        cfg.n_heads = std::max(cfg.n_heads, L.heads); cfg.n_kv_heads = std::max(cfg.n_kv_heads, L.kv_heads);
        cfg.head_dim = std::max(cfg.head_dim, L.dim); cfg.intermediate_size = std::max(cfg.intermediate_size, L.ff);
    }
    cfg.max_seq_len = 4096;
    return true;
}

// The rank of the WKV decay: rows of '<layer>.mix.w1'.
bool sizes_from_tensors(ModelConfig& cfg, const TensorShapeFn& shape_of, std::string& err) {
    for (int i = 0; i < cfg.n_layers; i++) {
        LayerSpec& L = cfg.layers[(size_t)i];
        if (L.mixer != MixerKind::WKV || L.wkv.decay_rank > 0) continue;
        const std::string name = "l" + std::to_string(i) + ".mix.w1";
        std::vector<int64_t> sh;
        if (!shape_of(name, sh) || sh.size() != 2 || sh[0] <= 0) { err = "tensor " + name + " is missing or not a matrix"; return false; }
        L.wkv.decay_rank = (int)sh[0];
    }
    return true;
}

std::vector<TensorBinding> tensors(const ModelConfig& cfg) {
    std::vector<TensorBinding> t;
    const int W = cfg.hidden_size;
    t.push_back({"embed", TensorSlot::EMBED, -1, cfg.vocab_size, W});
    if (cfg.bigram_buckets > 0) t.push_back({"bigram", TensorSlot::BIGRAM, -1, cfg.bigram_buckets + 1, W});
    t.push_back({"final.norm", TensorSlot::OUT_NORM, -1, 1, W});
    for (int i = 0; i < cfg.n_layers; i++) {
        const LayerSpec& L = cfg.layers[(size_t)i];
        const std::string p = "l" + std::to_string(i) + ".", q = p + "mix.";
        t.push_back({p + "norm1", TensorSlot::NORM1, i, 1, W});
        if (L.mixer == MixerKind::ATTN_LATENT) {
            const LatentSpec& A = L.latent;
            t.push_back({q + "q", TensorSlot::WQ, i, L.heads * (L.dim + A.rot_dim), W});
            t.push_back({q + "dkv", TensorSlot::W_DKV, i, A.kv_rank + A.rot_dim, W});
            t.push_back({q + "dkv.norm", TensorSlot::DKV_NORM, i, 1, A.kv_rank});
            if (L.dim > 0) t.push_back({q + "uk", TensorSlot::W_UK, i, L.heads * L.dim, A.kv_rank});
            t.push_back({q + "uv", TensorSlot::W_UV, i, L.heads * L.vdim, A.kv_rank});
            t.push_back({q + "o", TensorSlot::WO, i, W, L.heads * L.vdim});
        } else {
            const int n = L.heads * L.dim, rank = L.wkv.decay_rank;
            const char* blends[5] = {"mu.r", "mu.k", "mu.v", "mu.g", "mu.w"};
            for (int s = 0; s < 5; s++) t.push_back({q + blends[s], TensorSlot::WKV_MU, i, 1, W, s});
            t.push_back({q + "r", TensorSlot::WQ, i, n, W});
            t.push_back({q + "k", TensorSlot::WK, i, n, W});
            t.push_back({q + "v", TensorSlot::WV, i, n, W});
            t.push_back({q + "g", TensorSlot::WKV_G, i, n, W});
            t.push_back({q + "w1", TensorSlot::WKV_W1, i, rank, W});
            t.push_back({q + "w2", TensorSlot::WKV_W2, i, n, rank});
            t.push_back({q + "w0", TensorSlot::WKV_W0, i, 1, n});
            t.push_back({q + "u", TensorSlot::WKV_U, i, L.heads, L.dim});
            t.push_back({q + "norm", TensorSlot::WKV_NORM, i, 1, n});
            t.push_back({q + "o", TensorSlot::WO, i, W, n});
        }
        if (L.ff > 0 && L.ff_kind == FfKind::MLP) {
            t.push_back({p + "mlp.up", TensorSlot::UP, i, L.ff, W});
            t.push_back({p + "mlp.down", TensorSlot::DOWN, i, W, L.ff});
            t.push_back({p + "mlp.act", TensorSlot::FF_ACT, i, 1, 2});
        } else if (L.ff > 0) {
            t.push_back({p + "mlp.router", TensorSlot::ROUTER, i, L.experts, W});
            for (int e = 0; e < L.experts; e++) {
                const std::string x = p + "mlp.e" + std::to_string(e) + ".";
                t.push_back({x + "gate", TensorSlot::EXPERT_GATE, i, L.ff, W, e});
                t.push_back({x + "up", TensorSlot::EXPERT_UP, i, L.ff, W, e});
                t.push_back({x + "down", TensorSlot::EXPERT_DOWN, i, W, L.ff, e});
            }
            if (L.shared_ff > 0) {
                t.push_back({p + "mlp.shared.gate", TensorSlot::SHARED_GLU, i, L.shared_ff, W});
                t.push_back({p + "mlp.shared.up", TensorSlot::SHARED_UP, i, L.shared_ff, W});
                t.push_back({p + "mlp.shared.down", TensorSlot::SHARED_DOWN, i, W, L.shared_ff});
            }
        }
        t.push_back({p + "dwa", TensorSlot::DEPTH_AVG, i, 1, i + 2});
    }
    return t;
}

const ModelFamily kFamily = {"Fuvozen", config_from_json, tensors, sizes_from_tensors};

}  // namespace

const ModelFamily* fuvozen_family() { return &kFamily; }

}}  // namespace nt::b200
