#include "config/fifotar.h"

#include <cmath>

namespace illm {

namespace {
const Json& need_obj(const Json& d, const std::string& key, const std::string& where) {
    if (!d.is_object() || !d.has(key) || !d.at(key).is_object()) throw ConfigError("config.json: " + where + "'" + key + "' must be an object");
    return d.at(key);
}
bool given(const Json& d, const std::string& key) { return d.is_object() && d.has(key) && !d.at(key).is_null(); }
double need_number(const Json& d, const std::string& key, const std::string& where) {
    if (!d.is_object() || !d.has(key) || !d.at(key).is_number()) throw ConfigError("config.json: " + where + "'" + key + "' must be a number");
    return d.at(key).as_double();
}
double need_positive(const Json& d, const std::string& key, const std::string& where) {
    const double v = need_number(d, key, where);
    if (!(v > 0)) throw ConfigError("config.json: " + where + "'" + key + "' must be positive");
    return v;
}
Json obj(std::initializer_list<std::pair<const char*, Json>> kv) {
    Json o = Json::object();
    for (auto& p : kv) o.set(p.first, p.second);
    return o;
}
Json name_map(std::initializer_list<std::pair<const char*, const char*>> kv) {
    Json o = Json::object();
    for (auto& p : kv) o.set(p.first, std::string(p.second));
    return o;
}
}  // namespace

std::unique_ptr<ArchConfig> FifotarConfig::from_json(const Json& d) {
    std::unique_ptr<FifotarConfig> c(new FifotarConfig);
    c->raw = d;
    c->width = take_int(d, "width");
    c->vocab = take_int(d, "vocab");
    c->max_positions = take_int(d, "max_positions", 131072);
    c->norm_eps = need_positive(need_obj(d, "norm", ""), "eps", "norm: ");
    if (given(d, "embedding") && given(need_obj(d, "embedding", ""), "scale")) c->embedding_scale = need_number(d.at("embedding"), "scale", "embedding: ");
    if (given(d, "residual_mult")) c->residual_mult = need_number(d, "residual_mult", "");
    if (given(d, "logit_softcap")) c->logit_softcap = need_positive(d, "logit_softcap", "");
    if (c->width <= 0 || c->vocab <= 0 || c->max_positions <= 0) throw ConfigError("config.json: width, vocab and max_positions must be positive");
    if (!d.has("layers") || !d.at("layers").is_array() || d.at("layers").size() == 0)
        throw ConfigError("config.json: 'layers' must be a list with at least one layer");
    c->model_spec();        // every layer is checked now, not at the first use
    return std::unique_ptr<ArchConfig>(c.release());
}

ModelSpec FifotarConfig::model_spec() const {
    ModelSpec s;
    s.hidden_size = width;
    s.vocab_size = vocab;
    s.max_positions = max_positions;
    // RMS norm x / sqrt(mean(x^2) + eps) * w; behind a sublayer its output joins the stream times residual_mult
    auto norm = [&](double post_scale) {
        return PartSpec("rmsnorm", obj({{"size", width}, {"eps", norm_eps}, {"float32_weight", true}, {"post_scale", post_scale}, {"tensor", std::string("")}}));
    };
    const Json& layers = raw.at("layers");
    size_t i = 0;
    long long first_values = 0;          // the value width of the first layer that mixes values; 0 before it
    for (const Json& L : layers.items()) {
        const std::string where = "layer " + std::to_string(i) + ": ";
        if (!L.is_object()) throw ConfigError("config.json: " + where + "must be an object");
        const std::string type = take_string(L, "type", "");
        const Json& m = need_obj(L, "mixer", where);
        const bool has_mlp = given(L, "mlp");
        LayerSpec l;
        l.prefix = "l" + std::to_string(i) + ".";
        l.block = has_mlp ? "sandwich" : "sandwich_mixer";
        l.names = {{"mixer", "mix."}, {"ffn", "mlp."}, {"norm1", "norm1"}, {"norm1b", "norm1b"}};
        l.norms["norm1"] = norm(1.0);
        l.norms["norm1b"] = norm(residual_mult);
        if (has_mlp) {
            l.names["norm2"] = "norm2";
            l.names["norm2b"] = "norm2b";
            l.norms["norm2"] = norm(1.0);
            l.norms["norm2b"] = norm(residual_mult);
        }
        const long long heads = take_int(m, "heads"), dim = take_int(m, "dim"), vdim = take_int(m, "vdim");
        if (heads <= 0 || dim <= 0 || vdim <= 0) throw ConfigError("config.json: " + where + "heads, dim and vdim must be positive");
        auto kv_heads = [&]() {
            const long long g = take_int(m, "kv_heads", heads);
            if (g <= 0 || heads % g) throw ConfigError("config.json: " + where + "heads must be a multiple of kv_heads");
            return g;
        };
        if (type == "delta") {
            // the gated delta rule over a float32 state per head with one decay per head; short causal convolutions and silu on
            // q, k and v, unit q and k, q also times dim^(-1/2); a per-head unit norm with a shared weight and a silu gate
            const long long taps = take_int(m, "conv", 1);
            if (taps < 1) throw ConfigError("config.json: " + where + "conv must be at least 1");
            l.mixer = PartSpec("head_delta", obj({{"hidden_size", width}, {"n_heads", heads}, {"n_kv_heads", kv_heads()}, {"head_dim", dim}, {"v_head_dim", vdim},
                                                  {"conv", taps}, {"norm_eps", norm_eps}, {"q_scale", 1.0 / std::sqrt((double)dim)},
                                                  {"output_dtype", std::string("float32")},
                                                  {"names", name_map({{"q", "q"}, {"k", "k"}, {"v", "v"}, {"q_conv", "q.conv"}, {"k_conv", "k.conv"},
                                                                      {"v_conv", "v.conv"}, {"beta", "b"}, {"a_log", "A_log"}, {"norm", "norm"}, {"a", "a"},
                                                                      {"dt_bias", "dt_bias"}, {"gate", "g"}, {"o", "o"}})}}));
        } else if (type == "latent_attention") {
            // attention whose queries come out of a normed latent and whose keys and values are maps of a second one (the only
            // thing cached, beside one rotated key part that all heads share); all earlier positions; a sigmoid gate per head
            const long long q_rank = take_int(m, "q_rank"), kv_rank = take_int(m, "kv_rank"), rot_dim = take_int(m, "rot_dim", 0);
            if (q_rank <= 0 || kv_rank <= 0 || rot_dim < 0) throw ConfigError("config.json: " + where + "q_rank and kv_rank must be positive and rot_dim not negative");
            Json p = obj({{"hidden_size", width}, {"n_heads", heads}, {"head_dim", dim}, {"v_head_dim", vdim}, {"q_rank", q_rank}, {"kv_rank", kv_rank},
                          {"rot_head_dim", rot_dim}, {"scale", need_number(m, "scale", where)}, {"norm_eps", norm_eps},
                          {"out_gate", std::string("head_sigmoid")}, {"output_dtype", std::string("float32")},
                          {"names", name_map({{"q_down", "dq"}, {"q_norm", "dq.norm"}, {"q_up", "uq"}, {"kv_down", "dkv"}, {"kv_norm", "dkv.norm"}, {"k_up", "uk"},
                                              {"v_up", "uv"}, {"gate", "g"}, {"o", "o"}})}});
            if (rot_dim > 0) {
                const Json& rot = need_obj(m, "rot", where);
                const long long dims = take_int(rot, "dims", rot_dim);
                if (dims <= 0 || dims % 2 || dims > rot_dim) throw ConfigError("config.json: " + where + "rot.dims must be even and at most rot_dim");
                Json pos = obj({{"head_dim", rot_dim}, {"rot_dim", dims}, {"theta", need_positive(rot, "base", where + "rot: ")}, {"max_positions", max_positions}});
                if (given(rot, "scaling")) {
                    const Json& sc = need_obj(rot, "scaling", where + "rot: ");
                    const std::string at = where + "rot.scaling: ";
                    pos.set("scaling", obj({{"factor", need_positive(sc, "factor", at)}, {"original", need_positive(sc, "original", at)},
                                            {"fast", need_positive(sc, "fast", at)}, {"slow", need_positive(sc, "slow", at)}}));
                }
                p.set("position", PartSpec("rope_half", pos).to_json());
            }
            l.mixer = PartSpec("latent_attention", p);
        } else if (type == "attention") {
            // softmax attention without positions inside chunks of the sequence, capped scores, one added to the softmax
            // denominator, values mixed with the first such layer's, an element-wise sigmoid gate
            const long long kvh = kv_heads();
            long long chunk = 0;
            if (given(m, "mask")) {
                chunk = take_int(need_obj(m, "mask", where), "size");
                if (chunk < 1) throw ConfigError("config.json: " + where + "mask.size must be at least 1");
            }
            Json p = obj({{"hidden_size", width}, {"n_heads", heads}, {"n_kv_heads", kvh}, {"head_dim", dim}, {"v_head_dim", vdim}, {"chunk", chunk},
                          {"scale", need_number(m, "scale", where)}, {"norm_eps", norm_eps}, {"unit_sink", true}, {"out_gate", std::string("sigmoid")},
                          {"output_dtype", std::string("float32")}, {"position", PartSpec("none", Json::object()).to_json()},
                          {"names", name_map({{"q", "q"}, {"k", "k"}, {"v", "v"}, {"gate", "g"}, {"v_mix", "vmix"}, {"o", "o"}})}});
            if (given(m, "softcap")) p.set("softcap", need_positive(m, "softcap", where));
            if (take_bool(m, "v_mix", false)) {
                p.set("value_mix", std::string(first_values ? "mix" : "first"));
                if (first_values && first_values != kvh * vdim)
                    throw ConfigError("config.json: " + where + "layers that mix values must have as many value channels as the first of them");
                first_values = kvh * vdim;
            }
            l.mixer = PartSpec("attention", p);
        } else {
            throw ConfigError("config.json: " + where + "unknown type '" + type + "' (delta, latent_attention, attention)");
        }
        if (has_mlp) {
            const Json& mlp = need_obj(L, "mlp", where);
            const std::string kind = take_string(mlp, "kind", "dense");
            if (kind != "dense") throw ConfigError("config.json: " + where + "mlp.kind '" + kind + "' is not supported (dense)");
            l.ffn = PartSpec("gated_mlp", obj({{"hidden_size", width}, {"intermediate_size", take_int(mlp, "ff")}, {"activation", std::string("swish_clamped")},
                                               {"activation_limit", need_positive(mlp, "limit", where + "mlp: ")}, {"output_dtype", std::string("float32")},
                                               {"names", name_map({{"gate", "gate"}, {"up", "up"}, {"down", "down"}})}}));
        }
        s.layers.push_back(l);
        s.schedule.push_back(ScheduleEntry{(int)i, (int)i, true, false});
        i++;
    }
    s.embedding = PartSpec("embedding", obj({{"name", std::string("embed")}, {"tensor", std::string("")}, {"vocab_size", vocab}, {"hidden_size", width},
                                             {"scale", embedding_scale}}));
    s.final_norm = PartSpec("rmsnorm", obj({{"name", std::string("final.norm")}, {"tensor", std::string("")}, {"size", width}, {"eps", norm_eps},
                                            {"float32_weight", true}}));
    Json head = obj({{"name", std::string("head")}, {"tensor", std::string("")}, {"tied", true}, {"vocab_size", vocab}, {"hidden_size", width}});
    if (logit_softcap > 0) head.set("softcap", logit_softcap);
    s.head = PartSpec("lm_head", head);
    return s;
}

void register_fifotar_architecture() { register_architecture("Fifotar", &FifotarConfig::from_json, {"fifotar"}); }

}  // namespace illm
