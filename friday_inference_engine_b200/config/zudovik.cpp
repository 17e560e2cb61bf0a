// Zudovik: its config.json, checked and completed, and how it turns into parts.
//
// config.json is nested: "vocab", "width", "embedding": {"scale"}, "norm": {"eps"}, "layers": a list of {"type", "mixer", "mlp"}.
// Every size and constant comes from there.
//
// The model: token rows times a multiplier as a 32-bit residual stream; layers whose sublayers read the stream itself and
// whose results are RMS-normed before they join it; a mixer that is either linear attention with a constant decay per head
// ("lightning"), or causal softmax attention ("attention": grouped key/value heads, biased projections, one norm over all
// query heads and one over all key heads, rotation of neighbouring pairs, capped scores, a sink and a gate per head) that may
// read the keys and values of an earlier layer instead of making its own ("kv_from"); a dense feed-forward with a squared
// activation, or routed experts (softmax scores, a correction for the choice, experts that return their input, clipped gated
// units) with a gated expert that every token uses; or none; a final norm and a head of its own.
#include "friday/config.h"
#include "friday/parts.h"

namespace friday {

namespace {
const char* kName = "Zudovik";
constexpr double kGateSlope = 1.702;          // of the experts' gate: g sigmoid(1.702 g)

const Json& member(const Json& d, const std::string& key, const std::string& where) {
    const Json* v = d.is_object() ? d.find(key) : nullptr;
    if (!v || v->is_null()) throw ConfigError("config.json: " + where + "needs '" + key + "'");
    return *v;
}

const Json* optional(const Json& d, const std::string& key) {
    const Json* v = d.is_object() ? d.find(key) : nullptr;
    return v && !v->is_null() ? v : nullptr;
}

int64_t positive_int(const Json& d, const std::string& key, const std::string& where) {
    const Json& v = member(d, key, where);
    if (!v.is_int() || v.as_int() <= 0) throw ConfigError("config.json: " + where + "'" + key + "' must be a positive integer");
    return v.as_int();
}

double number(const Json& d, const std::string& key, const std::string& where) {
    const Json& v = member(d, key, where);
    if (!v.is_number()) throw ConfigError("config.json: " + where + "'" + key + "' must be a number");
    return v.as_double();
}

double positive(const Json& d, const std::string& key, const std::string& where) {
    const double v = number(d, key, where);
    if (!(v > 0)) throw ConfigError("config.json: " + where + "'" + key + "' must be positive");
    return v;
}

void check_lightning(const Json& m, const std::string& where) {
    const int64_t heads = positive_int(m, "heads", where);
    positive_int(m, "dim", where);
    positive_int(m, "vdim", where);
    const Json& d = member(m, "decay", where);
    if (!d.is_array() || (int64_t)d.size() != heads) throw ConfigError(format("config.json: %s'decay' must be a list of %lld numbers, one per head", where.c_str(), (long long)heads));
    for (size_t i = 0; i < d.size(); ++i)
        if (!d[i].is_number()) throw ConfigError("config.json: " + where + "'decay' must hold numbers");
}

void check_attention(const Json& m, const Json& layers, size_t index, const std::string& where) {
    const int64_t heads = positive_int(m, "heads", where), kv = positive_int(m, "kv_heads", where);
    if (heads % kv) throw ConfigError(format("config.json: %s%lld heads cannot share %lld key/value heads", where.c_str(), (long long)heads, (long long)kv));
    const int64_t dim = positive_int(m, "dim", where), vdim = positive_int(m, "vdim", where);
    number(m, "scale", where);
    if (optional(m, "softcap")) positive(m, "softcap", where);
    if (const Json* rot = optional(m, "rot")) {
        const std::string rw = where + "rot: ";
        if (!(number(*rot, "base", rw) > 1.0)) throw ConfigError("config.json: " + rw + "'base' must be greater than 1");
        const int64_t dims = positive_int(*rot, "dims", rw);
        if (dims > dim || dims % 2) throw ConfigError("config.json: " + rw + "'dims' must be even and at most the mixer's 'dim'");
    }
    const Json* from = optional(m, "kv_from");
    if (!from) return;
    // the layer whose keys and values are read: an earlier attention layer that makes its own, of the same key/value shape
    if (!from->is_int() || from->as_int() < 0 || from->as_int() >= (int64_t)index)
        throw ConfigError("config.json: " + where + "'kv_from' must name an earlier layer");
    const Json& other = layers[(size_t)from->as_int()];
    if (member(other, "type", where).as_string() != "attention" || optional(member(other, "mixer", where), "kv_from"))
        throw ConfigError("config.json: " + where + "'kv_from' must name an attention layer with keys and values of its own");
    const Json& om = other.at("mixer");
    if (om.at("kv_heads").as_int() != kv || om.at("dim").as_int() != dim || om.at("vdim").as_int() != vdim)
        throw ConfigError("config.json: " + where + "'kv_from' names a layer whose keys and values have another shape");
}

void check_unit(const Json& d, const std::string& where) {
    positive_int(d, "ff", where);
    positive(d, "limit", where);
}

void check_mlp(const Json& mlp, const std::string& where) {
    const std::string kind = member(mlp, "kind", where).as_string();
    if (kind == "dense") {
        positive_int(mlp, "ff", where);
        return;
    }
    if (kind != "moe") throw ConfigError("config.json: " + where + "feed-forward kind '" + kind + "' is not one this design has (dense, moe)");
    check_unit(member(mlp, "expert", where), where + "expert: ");
    const Json& router = member(mlp, "router", where);
    const std::string rw = where + "router: ";
    const int64_t experts = positive_int(router, "experts", rw), top = positive_int(router, "top", rw);
    int64_t identity = 0;
    if (const Json* id = optional(router, "identity")) {
        if (!id->is_int() || id->as_int() < 0) throw ConfigError("config.json: " + rw + "'identity' must be an integer that is not negative");
        identity = id->as_int();
    }
    if (top > experts + identity) throw ConfigError(format("config.json: %s%lld choices of %lld experts", rw.c_str(), (long long)top, (long long)(experts + identity)));
    if (const Json* shared = optional(mlp, "shared")) check_unit(*shared, where + "shared: ");
}

Json read_zudovik(const Json& d) {
    if (!d.is_object()) throw ConfigError("config.json: not an object");
    positive_int(d, "vocab", "");
    positive_int(d, "width", "");
    number(member(d, "embedding", ""), "scale", "embedding: ");
    positive(member(d, "norm", ""), "eps", "norm: ");
    const Json& layers = member(d, "layers", "");
    if (!layers.is_array() || layers.size() == 0) throw ConfigError("config.json: 'layers' must be a list of at least one layer");
    for (size_t i = 0; i < layers.size(); ++i) {
        const std::string where = format("layers[%zu]: ", i);
        const std::string type = member(layers[i], "type", where).as_string();
        const Json& mixer = member(layers[i], "mixer", where);
        if (type == "lightning") check_lightning(mixer, where + "mixer: ");
        else if (type == "attention") check_attention(mixer, layers, i, where + "mixer: ");
        else throw ConfigError("config.json: " + where + "mixer type '" + type + "' is not one this design has (lightning, attention)");
        if (const Json* mlp = optional(layers[i], "mlp")) check_mlp(*mlp, where + "mlp: ");
    }
    Json v = d;                                   // complete as given; the names the registry looks for are added
    Json a = Json::array();
    a.push(Json(kName));
    v.set("architectures", a);
    v.set("architecture", Json(kName));
    return v;
}

PartSpec norm_spec(double eps, const std::string& tensor_name) {
    Json p = Json::object();
    p.set("eps", Json(eps));
    p.set("weight_name", Json(tensor_name));
    return PartSpec("rmsnorm", p, "");
}

PartSpec lightning_spec(const Json& m, double eps) {
    Json p = Json::object();
    for (const char* k : {"heads", "dim", "vdim", "decay"}) p.set(k, m.at(k));
    p.set("eps", Json(eps));
    return PartSpec("decayed_linear_attention", p, "mix.");
}

PartSpec attention_spec(const Json& m, double eps) {
    Json p = Json::object();
    for (const char* k : {"heads", "kv_heads", "dim", "vdim", "scale"}) p.set(k, m.at(k));
    if (const Json* c = optional(m, "softcap")) p.set("softcap", *c);
    p.set("eps", Json(eps));
    p.set("qkv_bias", Json(true));
    p.set("qk_norm", Json("whole"));
    p.set("sink", Json(true));
    p.set("head_gate", Json(true));
    if (optional(m, "kv_from")) p.set("shared_kv", Json(true));
    PartSpec s("pooled_attention", p, "mix.");
    if (const Json* rot = optional(m, "rot")) {
        Json rp = Json::object();
        rp.set("base", rot->at("base"));
        rp.set("dims", rot->at("dims"));
        rp.set("layout", Json("neighbours"));
        s.parts["position"] = PartSpec("rotary_pairs", rp, "");
    } else {
        s.parts["position"] = PartSpec("none", Json::object(), "");
    }
    return s;
}

PartSpec mlp_spec(const Json& mlp) {
    Json p = Json::object();
    if (mlp.at("kind").as_string() == "dense") {
        p.set("inner", mlp.at("ff"));
        p.set("activation", Json("relu_squared"));
        return PartSpec("dense", p, "mlp.");
    }
    const Json& router = mlp.at("router");
    p.set("experts", router.at("experts"));
    p.set("top", router.at("top"));
    if (const Json* id = optional(router, "identity")) p.set("identity", *id);
    p.set("inner", mlp.at("expert").at("ff"));
    p.set("score", Json("softmax_biased"));
    p.set("router_bias", Json(false));
    p.set("choice_bias", Json("correction"));
    p.set("activation", Json("clipped"));
    p.set("slope", Json(kGateSlope));
    p.set("limit", mlp.at("expert").at("limit"));
    if (const Json* shared = optional(mlp, "shared")) {
        p.set("shared_inner", shared->at("ff"));
        p.set("shared_limit", shared->at("limit"));
        p.set("shared_gate", Json("shared.sg"));
    }
    return PartSpec("routed_experts", p, "mlp.");
}

ModelSpec zudovik_spec(const Json& c) {
    ModelSpec spec;
    spec.architecture = kName;
    spec.vocab_size = c.at("vocab").as_int();
    spec.width = c.at("width").as_int();
    spec.max_positions = (int64_t)1 << 30;            // nothing bounds a sequence but the cache
    spec.embedding = "embed";
    spec.embed_scale = c.at("embedding").at("scale").as_double();
    spec.head = "head";
    spec.residual_f32 = true;
    const double eps = c.at("norm").at("eps").as_double();
    spec.final_norm = norm_spec(eps, "final.norm");
    const Json& layers = c.at("layers");
    for (size_t i = 0; i < layers.size(); ++i) {
        const Json& L = layers[i];
        PartSpec block("sandwich", Json::object(), format("l%zu.", i));
        block.parts["norm1"] = PartSpec("identity");
        block.parts["norm1b"] = norm_spec(eps, "norm1");
        const bool lightning = L.at("type").as_string() == "lightning";
        block.parts["mixer"] = lightning ? lightning_spec(L.at("mixer"), eps) : attention_spec(L.at("mixer"), eps);
        if (const Json* mlp = optional(L, "mlp")) {
            block.parts["norm2"] = PartSpec("identity");
            block.parts["norm2b"] = norm_spec(eps, "norm2");
            block.parts["feed_forward"] = mlp_spec(*mlp);
        } else {
            spec.ignorable.push_back(format("l%zu.norm2", i));      // a checkpoint may carry it all the same
        }
        spec.layers.push_back(block);
        LayerCall call;
        call.layer = (int)i;
        call.cache = (int)i;
        if (const Json* from = lightning ? nullptr : optional(L.at("mixer"), "kv_from")) {
            call.cache = (int)from->as_int();                        // the entry that the other layer fills
            call.write = false;
        }
        spec.program.push_back(call);
    }
    return spec;
}

struct RegisterZudovik {
    RegisterZudovik() { register_architecture({kName, read_zudovik, zudovik_spec}); }
} register_zudovik;
}  // namespace

}  // namespace friday
