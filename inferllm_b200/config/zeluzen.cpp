#include "config/zeluzen.h"

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

std::unique_ptr<ArchConfig> ZeluzenConfig::from_json(const Json& d) {
    std::unique_ptr<ZeluzenConfig> c(new ZeluzenConfig);
    c->raw = d;
    c->width = take_int(d, "width");
    c->vocab = take_int(d, "vocab");
    c->max_positions = take_int(d, "max_positions", 131072);
    c->norm_eps = need_positive(need_obj(d, "norm", ""), "eps", "norm: ");
    if (c->width <= 0 || c->vocab <= 0 || c->max_positions <= 0) throw ConfigError("config.json: width, vocab and max_positions must be positive");
    if (!d.has("layers") || !d.at("layers").is_array() || d.at("layers").size() == 0)
        throw ConfigError("config.json: 'layers' must be a list with at least one layer");
    c->model_spec();        // every layer is checked now, not at the first use
    return std::unique_ptr<ArchConfig>(c.release());
}

ModelSpec ZeluzenConfig::model_spec() const {
    ModelSpec s;
    s.hidden_size = width;
    s.vocab_size = vocab;
    s.max_positions = max_positions;
    // RMS norm x / sqrt(mean(x^2) + eps) * w
    const PartSpec norm("rmsnorm", obj({{"size", width}, {"eps", norm_eps}, {"float32_weight", true}, {"tensor", std::string("")}}));
    const Json& layers = raw.at("layers");
    struct KeysValues { long long kv_heads, dim, vdim; };       // of the layers that have keys and values of their own
    std::map<long long, KeysValues> own;
    size_t i = 0;
    for (const Json& L : layers.items()) {
        const std::string where = "layer " + std::to_string(i) + ": ";
        if (!L.is_object()) throw ConfigError("config.json: " + where + "must be an object");
        const std::string type = take_string(L, "type", "");
        const Json& m = need_obj(L, "mixer", where);
        const bool has_mlp = given(L, "mlp");
        LayerSpec l;
        l.prefix = "l" + std::to_string(i) + ".";
        l.block = has_mlp ? "outnorm" : "outnorm_mixer";
        l.names = {{"mixer", "mix."}, {"ffn", "mlp."}, {"norm1", "norm1"}};
        l.norms["norm1"] = norm;
        if (has_mlp) {
            l.names["norm2"] = "norm2";
            l.norms["norm2"] = norm;
        }
        const long long heads = take_int(m, "heads"), dim = take_int(m, "dim");
        if (heads <= 0 || dim <= 0) throw ConfigError("config.json: " + where + "heads and dim must be positive");
        int cache_entry = (int)i;
        bool writes = true;
        if (type == "wkv") {
            // a recurrence over a float32 state per head with a decay per key channel that the token makes itself; five blends
            // of the token's and the previous token's row feed its projections; a per-head unit norm, a weight, a silu gate
            l.mixer = PartSpec("wkv", obj({{"hidden_size", width}, {"n_heads", heads}, {"head_dim", dim}, {"norm_eps", norm_eps},
                                           {"output_dtype", std::string("float32")},
                                           {"names", name_map({{"r", "r"}, {"k", "k"}, {"v", "v"}, {"gate", "g"}, {"mu", "mu."}, {"mu_gate", "g"}, {"w1", "w1"},
                                                               {"w2", "w2"}, {"w0", "w0"}, {"bonus", "u"}, {"norm", "norm"}, {"o", "o"}})}}));
            // the inner size of the decay's map is the file's (the shape of w1); a model made from random numbers names it
            if (given(m, "decay_rank")) l.mixer.params.set("decay_rank", take_int(m, "decay_rank"));
        } else if (type == "attention") {
            // softmax attention inside chunks of the sequence, one added to the softmax denominator; an RMS norm per query and
            // key head in front of an interleaved-pair rotation
            const long long kvh = take_int(m, "kv_heads", heads), vdim = take_int(m, "vdim", dim);
            if (kvh <= 0 || heads % kvh || vdim <= 0) throw ConfigError("config.json: " + where + "heads must be a multiple of kv_heads and vdim positive");
            long long chunk = 0;
            if (given(m, "mask")) {
                chunk = take_int(need_obj(m, "mask", where), "size");
                if (chunk < 1) throw ConfigError("config.json: " + where + "mask.size must be at least 1");
            }
            Json p = obj({{"hidden_size", width}, {"n_heads", heads}, {"n_kv_heads", kvh}, {"head_dim", dim}, {"v_head_dim", vdim}, {"chunk", chunk},
                          {"scale", need_number(m, "scale", where)}, {"norm_eps", norm_eps}, {"unit_sink", true}, {"qk_norm", std::string("head")},
                          {"output_dtype", std::string("float32")},
                          {"names", name_map({{"q", "q"}, {"k", "k"}, {"v", "v"}, {"q_norm", "q.norm"}, {"k_norm", "k.norm"}, {"o", "o"}})}});
            long long dims = 0;
            if (given(m, "rot")) dims = take_int(need_obj(m, "rot", where), "dims", dim);
            if (dims > 0) {
                const Json& rot = m.at("rot");
                if (dims % 2 || dims > dim) throw ConfigError("config.json: " + where + "rot.dims must be even and at most dim");
                Json pos = obj({{"head_dim", dim}, {"rot_dim", dims}, {"theta", need_positive(rot, "base", where + "rot: ")}, {"max_positions", max_positions}});
                if (given(rot, "scaling")) {
                    const Json& sc = need_obj(rot, "scaling", where + "rot: ");
                    const std::string at = where + "rot.scaling: ";
                    pos.set("scaling", obj({{"factor", need_positive(sc, "factor", at)}, {"original", need_positive(sc, "original", at)},
                                            {"low", need_positive(sc, "low", at)}, {"high", need_positive(sc, "high", at)}}));
                }
                p.set("position", PartSpec("rope_pairs", pos).to_json());
            } else {
                p.set("position", PartSpec("none", Json::object()).to_json());
            }
            if (given(m, "kv_from")) {
                const long long j = take_int(m, "kv_from");
                auto it = own.find(j);
                if (it == own.end()) throw ConfigError("config.json: " + where + "kv_from must name an earlier attention layer with keys and values of its own");
                if (it->second.kv_heads != kvh || it->second.dim != dim || it->second.vdim != vdim)
                    throw ConfigError("config.json: " + where + "kv_from: the two layers' key and value heads differ");
                p.set("own_kv", false);
                cache_entry = (int)j;
                writes = false;
            } else {
                own[(long long)i] = KeysValues{kvh, dim, vdim};
            }
            l.mixer = PartSpec("attention", p);
        } else {
            throw ConfigError("config.json: " + where + "unknown type '" + type + "' (wkv, attention)");
        }
        if (has_mlp) {
            const Json& mlp = need_obj(L, "mlp", where);
            const std::string kind = take_string(mlp, "kind", "dense");
            if (kind == "dense") {
                l.ffn = PartSpec("gated_mlp", obj({{"hidden_size", width}, {"intermediate_size", take_int(mlp, "ff")}, {"activation", std::string("silu")},
                                                   {"output_dtype", std::string("float32")},
                                                   {"names", name_map({{"gate", "gate"}, {"up", "up"}, {"down", "down"}})}}));
            } else if (kind == "moe") {
                // experts without a gate, the square of relu; scores are a softmax over all experts, the identity experts (whose
                // output is their input) among them; a correction in the choice only; the weights are the scores themselves
                const Json& r = need_obj(mlp, "router", where + "mlp: ");
                l.ffn = PartSpec("routed_mlp", obj({{"hidden_size", width}, {"intermediate_size", take_int(need_obj(mlp, "expert", where + "mlp: "), "ff")},
                                                    {"experts", take_int(r, "experts")}, {"identity_experts", take_int(r, "identity", 0)}, {"top", take_int(r, "top")},
                                                    {"expert_kind", std::string("plain")}, {"activation", std::string("relu_squared")},
                                                    {"scoring", std::string("softmax_all")}, {"choice_correction", true}, {"renormalize", false},
                                                    {"names", name_map({{"router", "router"}, {"correction", "correction"}, {"expert", "e"}, {"up", "up"},
                                                                        {"down", "down"}})}}));
            } else {
                throw ConfigError("config.json: " + where + "mlp.kind '" + kind + "' is not supported (dense, moe)");
            }
        }
        s.layers.push_back(l);
        s.schedule.push_back(ScheduleEntry{(int)i, cache_entry, writes, false});
        i++;
    }
    s.embedding = PartSpec("embedding", obj({{"name", std::string("embed")}, {"tensor", std::string("")}, {"vocab_size", vocab}, {"hidden_size", width},
                                             {"norm", obj({{"tensor", std::string(".norm")}, {"eps", norm_eps}})}}));
    s.final_norm = PartSpec("rmsnorm", obj({{"name", std::string("final.norm")}, {"tensor", std::string("")}, {"size", width}, {"eps", norm_eps},
                                            {"float32_weight", true}}));
    s.head = PartSpec("lm_head", obj({{"name", std::string("head")}, {"tensor", std::string("")}, {"tied", false}, {"vocab_size", vocab}, {"hidden_size", width}}));
    return s;
}

void register_zeluzen_architecture() { register_architecture("Zeluzen", &ZeluzenConfig::from_json, {"zeluzen"}); }

}  // namespace illm
