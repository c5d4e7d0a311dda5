// tibelix.cpp — the Tibelix family: a decoder with a norm in front of and behind each sublayer (BlockForm::SANDWICH, gains stored around zero) whose
// layers, in any order the configuration lists, mix tokens by
//   "attention":        grouped-query attention without rotation: queries and keys over their root mean square per head (QKNorm::UNIT), a
//                       position-dependent query multiplier ("q_temp", LayerSpec::q_temp), scores minus a per-head slope times the distance
//                       (distance_bias), a softmax with one more 1 in its denominator (unit_sink) and one output gate per head; "kv_from" names an
//                       earlier attention layer whose cache rows the layer reads;
//   "latent_attention": low-rank attention with a query latent (MixerKind::ATTN_LATENT), interleaved rotary pairs with the long-context blend
//                       ("rot.scaling") and an output gate per channel; or
//   "mlstm":            the matrix memory with exponential gates (MixerKind::MLSTM, MlstmSpec).
// The feed-forward is W_down relu(W_up h)^2 (FfKind::MLP), a mixture of SiLU-gated experts chosen by the softmax over all of them, inside the groups
// with the largest score, weights divided by their sum (FfKind::MOE_GLU, RouteSpec), with an optional gated shared expert; or absent ("mlp": null).
// The head is the embedding table.  Every size and constant that varies between models of the family is read from config.json; an absent
// "q_temp", "rot", "rot.scaling", "router.groups" and "shared" switch their mechanism off.
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
template <typename F> bool need_float(const Json& o, const char* key, F& out, std::string& err, const std::string& where) {
    const Json& v = o.at(key);
    if (!v.is_number()) { err = where + ": \"" + key + "\" is missing or not a number"; return false; }
    out = (F)v.number_or(0.0);
    return true;
}

bool attention_from_json(const Json& m, LayerSpec& L, const ModelConfig& cfg, size_t i, std::string& err, const std::string& where) {
    L.mixer = MixerKind::ATTN_WINDOW;          // window 0: every earlier position is visible
    L.qk_norm = QKNorm::UNIT;
    L.distance_bias = true; L.unit_sink = true; L.out_gate = OutGate::PER_HEAD;
    if (!need_int(m, "heads", L.heads, err, where) || !need_int(m, "kv_heads", L.kv_heads, err, where) || !need_int(m, "dim", L.dim, err, where) ||
        !need_int(m, "vdim", L.vdim, err, where) || !need_float(m, "scale", L.scale, err, where)) return false;
    if (L.heads <= 0 || L.kv_heads <= 0 || L.heads % L.kv_heads || L.dim <= 0 || L.vdim <= 0) { err = where + ": invalid head sizes (heads % kv_heads == 0)"; return false; }
    if (m.has("q_temp") && m.at("q_temp").is_object()) {
        const Json& t = m.at("q_temp");
        if (!need_float(t, "coef", L.q_temp.coef, err, where + ".q_temp") || !need_float(t, "every", L.q_temp.every, err, where + ".q_temp")) return false;
        if (!(L.q_temp.every > 0.0)) { err = where + ": q_temp.every must be positive"; return false; }
    }
    if (m.has("kv_from") && m.at("kv_from").is_number()) {
        L.kv_from = (int)m.at("kv_from").int_or(-1);
        if (L.kv_from < 0 || L.kv_from >= (int)i) { err = where + ": \"kv_from\" must name an earlier layer"; return false; }
        const LayerSpec& J = cfg.layers[(size_t)L.kv_from];
        if (J.mixer != MixerKind::ATTN_WINDOW || J.kv_from >= 0) { err = where + ": \"kv_from\" must name an attention layer that has its own keys and values"; return false; }
        if (J.kv_heads != L.kv_heads || J.dim != L.dim || J.vdim != L.vdim) { err = where + ": \"kv_from\" layer has other key / value heads"; return false; }
    }
    return true;
}

bool latent_from_json(const Json& m, LayerSpec& L, std::string& err, const std::string& where) {
    L.mixer = MixerKind::ATTN_LATENT;
    L.kv_heads = 1;
    L.out_gate = OutGate::PER_CHANNEL;
    if (!need_int(m, "heads", L.heads, err, where) || !need_int(m, "dim", L.dim, err, where) || !need_int(m, "vdim", L.vdim, err, where) ||
        !need_int(m, "rot_dim", L.latent.rot_dim, err, where) || !need_int(m, "q_rank", L.latent.q_rank, err, where) ||
        !need_int(m, "kv_rank", L.latent.kv_rank, err, where) || !need_float(m, "scale", L.scale, err, where)) return false;
    if (L.heads <= 0 || L.dim <= 0 || L.vdim <= 0 || L.latent.rot_dim < 0 || L.latent.q_rank <= 0 || L.latent.kv_rank <= 0) { err = where + ": invalid mixer sizes"; return false; }
    if (m.has("rot") && m.at("rot").is_object()) {
        const Json& r = m.at("rot");
        if (!need_int(r, "dims", L.rot.dims, err, where + ".rot") || !need_float(r, "base", L.rot.base, err, where + ".rot")) return false;
        if (L.rot.dims < 0 || L.rot.dims > L.latent.rot_dim || (L.rot.dims & 1) || !(L.rot.base > 0.0)) { err = where + ": rot.dims must be even and at most rot_dim"; return false; }
        if (r.has("scaling") && r.at("scaling").is_object()) {
            const Json& c = r.at("scaling");
            const std::string w = where + ".rot.scaling";
            if (!need_float(c, "factor", L.rot.factor, err, w) || !need_float(c, "original", L.rot.original, err, w) || !need_float(c, "fast", L.rot.fast, err, w) ||
                !need_float(c, "slow", L.rot.slow, err, w)) return false;
            if (!(L.rot.factor > 0.f) || !(L.rot.original > 0.f) || !(L.rot.fast > 0.f) || !(L.rot.slow > 0.f) || L.rot.base == 1.0) { err = w + ": its numbers must be positive"; return false; }
        }
    }
    return true;
}

bool mlstm_from_json(const Json& m, LayerSpec& L, std::string& err, const std::string& where) {
    L.mixer = MixerKind::MLSTM;
    L.out_gate = OutGate::PER_CHANNEL;
    if (!need_int(m, "heads", L.heads, err, where) || !need_int(m, "dim", L.dim, err, where) || !need_int(m, "vdim", L.vdim, err, where) ||
        !need_float(m, "gate_cap", L.mlstm.gate_cap, err, where)) return false;
    L.kv_heads = L.heads;
    if (L.heads <= 0 || L.dim <= 0 || L.vdim <= 0 || !(L.mlstm.gate_cap > 0.f)) { err = where + ": invalid mixer sizes (gate_cap > 0)"; return false; }
    return true;
}

bool experts_from_json(const Json& mlp, LayerSpec& L, std::string& err, const std::string& where) {
    L.ff_kind = FfKind::MOE_GLU; L.act = GluAct::SILU;
    L.route.all = true; L.route.renorm = true;
    const Json& r = mlp.at("router");
    if (!need_int(mlp.at("expert"), "ff", L.ff, err, where + ".expert") || !need_int(r, "experts", L.experts, err, where + ".router") || !need_int(r, "top", L.top, err, where + ".router"))
        return false;
    if (L.ff <= 0 || L.experts <= 0 || L.top <= 0 || L.top > L.experts || L.experts > 256) { err = where + ": invalid expert sizes (1 <= top <= experts <= 256)"; return false; }
    if (r.has("groups") && r.at("groups").is_object()) {
        if (!need_int(r.at("groups"), "count", L.route.groups, err, where + ".router.groups") || !need_int(r.at("groups"), "keep", L.route.keep, err, where + ".router.groups")) return false;
        if (L.route.groups <= 0 || L.experts % L.route.groups || L.route.keep <= 0 || L.route.keep > L.route.groups || L.route.keep * (L.experts / L.route.groups) < L.top) {
            err = where + ": invalid expert groups (experts % count == 0, 1 <= keep <= count, the kept groups must hold at least top experts)"; return false;
        }
    }
    if (mlp.has("shared") && mlp.at("shared").is_object()) {
        L.shared_glu = true;
        if (!need_int(mlp.at("shared"), "ff", L.shared_ff, err, where + ".shared") || L.shared_ff <= 0) { if (err.empty()) err = where + ": invalid shared.ff"; return false; }
    }
    return true;
}

bool config_from_json(const Json& root, ModelConfig& cfg, std::string& err) {
    if (!need_int(root, "vocab", cfg.vocab_size, err, "config") || !need_int(root, "width", cfg.hidden_size, err, "config")) return false;
    if (!need_float(root.at("norm"), "eps", cfg.norm_eps, err, "config.norm")) return false;
    if (cfg.vocab_size <= 0 || cfg.hidden_size <= 0) { err = "config: invalid vocab / width"; return false; }
    cfg.norm_gain_offset = 1.0f;
    cfg.tied_head = true;
    const Json& layers = root.at("layers");
    if (!layers.is_array() || layers.arr.empty()) { err = "config: \"layers\" must be a non-empty list"; return false; }
    cfg.n_layers = (int)layers.arr.size();
    cfg.model_name = "tibelix";
    cfg.bos_token_id = -1; cfg.eos_token_id = -1;
    for (size_t i = 0; i < layers.arr.size(); i++) {
        const Json& e = layers.arr[i];
        const std::string where = "config.layers[" + std::to_string(i) + "]";
        LayerSpec L;
        L.form = BlockForm::SANDWICH;
        const std::string type = e.at("type").string_or("");
        const Json& m = e.at("mixer");
        if (!m.is_object()) { err = where + ": \"mixer\" is missing"; return false; }
        if (type == "attention") { if (!attention_from_json(m, L, cfg, i, err, where)) return false; }
        else if (type == "latent_attention") { if (!latent_from_json(m, L, err, where)) return false; }
        else if (type == "mlstm") { if (!mlstm_from_json(m, L, err, where)) return false; }
        else { err = where + ": mixer type \"" + type + "\" is not part of this family"; return false; }
        const Json& mlp = e.at("mlp");
        if (mlp.is_null()) L.ff = 0;
        else {
            const std::string kind = mlp.at("kind").string_or("");
            if (kind == "dense") {
                L.ff_kind = FfKind::MLP; L.act = GluAct::RELU2;
                if (!need_int(mlp, "ff", L.ff, err, where + ".mlp") || L.ff <= 0) { if (err.empty()) err = where + ": invalid ff"; return false; }
            } else if (kind == "moe") { if (!experts_from_json(mlp, L, err, where + ".mlp")) return false; }
            else { err = where + ": feed-forward kind \"" + kind + "\" is not part of this family"; return false; }
        }
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

std::vector<TensorBinding> tensors(const ModelConfig& cfg) {
    std::vector<TensorBinding> t;
    const int W = cfg.hidden_size;
    t.push_back({"embed", TensorSlot::EMBED, -1, cfg.vocab_size, W});
    t.push_back({"final.norm", TensorSlot::OUT_NORM, -1, 1, W});
    for (int i = 0; i < cfg.n_layers; i++) {
        const LayerSpec& L = cfg.layers[(size_t)i];
        const std::string p = "l" + std::to_string(i) + ".", q = p + "mix.", f = p + "mlp.";
        const int H = L.heads, D = L.dim, V = L.vdim;
        t.push_back({p + "norm1", TensorSlot::NORM1, i, 1, W});
        t.push_back({p + "norm1b", TensorSlot::NORM1B, i, 1, W});
        if (L.mixer == MixerKind::ATTN_LATENT) {
            const LatentSpec& A = L.latent;
            t.push_back({q + "dq", TensorSlot::W_DQ, i, A.q_rank, W});
            t.push_back({q + "dq.norm", TensorSlot::DQ_NORM, i, 1, A.q_rank});
            t.push_back({q + "uq", TensorSlot::W_UQ, i, H * (D + A.rot_dim), A.q_rank});
            t.push_back({q + "dkv", TensorSlot::W_DKV, i, A.kv_rank + A.rot_dim, W});
            t.push_back({q + "dkv.norm", TensorSlot::DKV_NORM, i, 1, A.kv_rank});
            t.push_back({q + "uk", TensorSlot::W_UK, i, H * D, A.kv_rank});
            t.push_back({q + "uv", TensorSlot::W_UV, i, H * V, A.kv_rank});
        } else {
            t.push_back({q + "q", TensorSlot::WQ, i, H * D, W});
            if (L.kv_from < 0) {
                t.push_back({q + "k", TensorSlot::WK, i, L.kv_heads * D, W});
                t.push_back({q + "v", TensorSlot::WV, i, L.kv_heads * V, W});
            }
        }
        if (L.mixer == MixerKind::MLSTM) {
            t.push_back({q + "i", TensorSlot::MLSTM_I, i, H, W});
            t.push_back({q + "i.b", TensorSlot::MLSTM_IB, i, 1, H});
            t.push_back({q + "f", TensorSlot::MLSTM_F, i, H, W});
            t.push_back({q + "f.b", TensorSlot::MLSTM_FB, i, 1, H});
            t.push_back({q + "norm", TensorSlot::MLSTM_NORM, i, 1, H * V});
        }
        t.push_back({q + "g", TensorSlot::OUT_GATE, i, L.out_gate == OutGate::PER_HEAD ? H : H * V, W});
        t.push_back({q + "o", TensorSlot::WO, i, W, H * V});
        if (L.ff == 0) continue;
        t.push_back({p + "norm2", TensorSlot::NORM2, i, 1, W});
        t.push_back({p + "norm2b", TensorSlot::NORM2B, i, 1, W});
        if (L.ff_kind == FfKind::MLP) {
            t.push_back({f + "up", TensorSlot::UP, i, L.ff, W});
            t.push_back({f + "down", TensorSlot::DOWN, i, W, L.ff});
            continue;
        }
        t.push_back({f + "router", TensorSlot::ROUTER, i, L.experts, W});
        for (int e = 0; e < L.experts; e++) {
            const std::string x = f + "e" + std::to_string(e) + ".";
            t.push_back({x + "gate", TensorSlot::EXPERT_GATE, i, L.ff, W, e});
            t.push_back({x + "up", TensorSlot::EXPERT_UP, i, L.ff, W, e});
            t.push_back({x + "down", TensorSlot::EXPERT_DOWN, i, W, L.ff, e});
        }
        if (L.shared_ff > 0) {
            t.push_back({f + "shared.gate", TensorSlot::SHARED_GLU, i, L.shared_ff, W});
            t.push_back({f + "shared.up", TensorSlot::SHARED_UP, i, L.shared_ff, W});
            t.push_back({f + "shared.down", TensorSlot::SHARED_DOWN, i, W, L.shared_ff});
        }
    }
    return t;
}

const ModelFamily kFamily = {"Tibelix", config_from_json, tensors};

}  // namespace

const ModelFamily* tibelix_family() { return &kFamily; }

}}  // namespace nt::b200
