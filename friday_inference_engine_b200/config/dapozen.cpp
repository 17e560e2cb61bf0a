// Dapozen: its config.json, checked and completed, and how it turns into parts.
//
// config.json is nested: "vocab", "width", "embedding": {"scale"}, "norm": {"eps"}, "layers": a list of {"type", "mixer", "mlp"}, and optionally
// "loop": {"start", "stop", "times"} and "logit_softcap".  Every size and constant comes from there.
//
// The model: token rows times a multiplier as a 32-bit residual stream; layers with an RMS norm before and after each sublayer,
// where the layers loop.start .. loop.stop-1 run loop.times times in a row with the same weights and a cache entry of their own each time; a
// mixer that is either softmax attention within runs of positions ("attention": grouped key/value heads, biased projections, a short
// convolution over time on queries, keys and values, rotation of neighbouring pairs, then heads divided by their root mean square, a sigmoid
// gate per channel) or state space duality ("mamba2"); a dense gated feed-forward, or experts that a table gives each token id, with clipped
// gated units, beside one that every token uses; or none; a final norm and a head of its own whose logits are capped.
#include "friday/config.h"
#include "friday/parts.h"

namespace friday {

namespace {
const char* kName = "Dapozen";
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

void check_attention(const Json& m, const std::string& where) {
    const int64_t heads = positive_int(m, "heads", where), kv = positive_int(m, "kv_heads", where);
    if (heads % kv) throw ConfigError(format("config.json: %s%lld heads cannot share %lld key/value heads", where.c_str(), (long long)heads, (long long)kv));
    const int64_t dim = positive_int(m, "dim", where);
    positive_int(m, "vdim", where);
    positive_int(m, "conv", where);
    number(m, "scale", where);
    if (const Json* rot = optional(m, "rot")) {
        const std::string rw = where + "rot: ";
        if (!(number(*rot, "base", rw) > 1.0)) throw ConfigError("config.json: " + rw + "'base' must be greater than 1");
        const int64_t dims = positive_int(*rot, "dims", rw);
        if (dims > dim || dims % 2) throw ConfigError("config.json: " + rw + "'dims' must be even and at most the mixer's 'dim'");
    }
    if (const Json* mask = optional(m, "mask")) positive_int(*mask, "size", where + "mask: ");
}

void check_mamba2(const Json& m, const std::string& where) {
    const int64_t heads = positive_int(m, "heads", where), groups = positive_int(m, "groups", where);
    if (heads % groups) throw ConfigError(format("config.json: %s%lld heads cannot share %lld groups", where.c_str(), (long long)heads, (long long)groups));
    const int64_t inner = heads * positive_int(m, "vdim", where), parts = positive_int(m, "norm_groups", where);
    if (inner % parts) throw ConfigError(format("config.json: %sa norm over %lld channels in %lld equal parts", where.c_str(), (long long)inner, (long long)parts));
    positive_int(m, "state", where);
    positive_int(m, "conv", where);
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
    if (top > experts) throw ConfigError(format("config.json: %s%lld choices of %lld experts", rw.c_str(), (long long)top, (long long)experts));
    if (const Json* shared = optional(mlp, "shared")) check_unit(*shared, where + "shared: ");
}

Json read_dapozen(const Json& d) {
    if (!d.is_object()) throw ConfigError("config.json: not an object");
    positive_int(d, "vocab", "");
    positive_int(d, "width", "");
    number(member(d, "embedding", ""), "scale", "embedding: ");
    positive(member(d, "norm", ""), "eps", "norm: ");
    if (optional(d, "logit_softcap")) positive(d, "logit_softcap", "");
    const Json& layers = member(d, "layers", "");
    if (!layers.is_array() || layers.size() == 0) throw ConfigError("config.json: 'layers' must be a list of at least one layer");
    for (size_t i = 0; i < layers.size(); ++i) {
        const std::string where = format("layers[%zu]: ", i);
        const std::string type = member(layers[i], "type", where).as_string();
        const Json& mixer = member(layers[i], "mixer", where);
        if (type == "attention") check_attention(mixer, where + "mixer: ");
        else if (type == "mamba2") check_mamba2(mixer, where + "mixer: ");
        else throw ConfigError("config.json: " + where + "mixer type '" + type + "' is not one this design has (attention, mamba2)");
        if (const Json* mlp = optional(layers[i], "mlp")) check_mlp(*mlp, where + "mlp: ");
    }
    if (const Json* loop = optional(d, "loop")) {
        const Json& a = member(*loop, "start", "loop: ");
        const Json& b = member(*loop, "stop", "loop: ");
        positive_int(*loop, "times", "loop: ");
        if (!a.is_int() || !b.is_int() || a.as_int() < 0 || b.as_int() <= a.as_int() || b.as_int() > (int64_t)layers.size())
            throw ConfigError(format("config.json: loop: 0 <= start < stop <= %zu layers", layers.size()));
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

PartSpec attention_spec(const Json& m, double eps) {
    Json p = Json::object();
    for (const char* k : {"heads", "kv_heads", "dim", "vdim", "scale", "conv"}) p.set(k, m.at(k));
    if (const Json* mask = optional(m, "mask")) p.set("chunk", mask->at("size"));
    p.set("eps", Json(eps));
    p.set("qkv_bias", Json(true));
    p.set("qk_norm", Json("unit"));
    p.set("gate", Json(true));
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

PartSpec mamba2_spec(const Json& m, double eps) {
    Json p = Json::object();
    for (const char* k : {"heads", "vdim", "state", "groups", "norm_groups", "conv"}) p.set(k, m.at(k));
    p.set("eps", Json(eps));
    return PartSpec("state_space_dual", p, "mix.");
}

PartSpec mlp_spec(const Json& mlp, int64_t vocab) {
    Json p = Json::object();
    if (mlp.at("kind").as_string() == "dense") {
        p.set("inner", mlp.at("ff"));
        Json names = Json::object();
        for (const char* n : {"gate", "up", "down"}) names.set(n, Json(n));
        p.set("names", names);
        return PartSpec("swiglu", p, "mlp.");
    }
    const Json& router = mlp.at("router");
    p.set("experts", router.at("experts"));
    p.set("top", router.at("top"));
    p.set("inner", mlp.at("expert").at("ff"));
    p.set("score", Json("table"));
    p.set("vocab", Json(vocab));
    p.set("router_bias", Json(false));
    p.set("activation", Json("clipped"));
    p.set("slope", Json(kGateSlope));
    p.set("limit", mlp.at("expert").at("limit"));
    if (const Json* shared = optional(mlp, "shared")) {
        p.set("shared_inner", shared->at("ff"));
        p.set("shared_limit", shared->at("limit"));
    }
    return PartSpec("routed_experts", p, "mlp.");
}

ModelSpec dapozen_spec(const Json& c) {
    ModelSpec spec;
    spec.architecture = kName;
    spec.vocab_size = c.at("vocab").as_int();
    spec.width = c.at("width").as_int();
    spec.max_positions = (int64_t)1 << 30;            // nothing bounds a sequence but the cache
    spec.embedding = "embed";
    spec.embed_scale = c.at("embedding").at("scale").as_double();
    spec.head = "head";
    if (const Json* cap = optional(c, "logit_softcap")) spec.logit_softcap = cap->as_double();
    spec.residual_f32 = true;
    const double eps = c.at("norm").at("eps").as_double();
    spec.final_norm = norm_spec(eps, "final.norm");
    const Json& layers = c.at("layers");
    const int64_t n = (int64_t)layers.size();
    for (int64_t i = 0; i < n; ++i) {
        const Json& L = layers[(size_t)i];
        PartSpec block("sandwich", Json::object(), format("l%lld.", (long long)i));
        block.parts["norm1"] = norm_spec(eps, "norm1");
        block.parts["norm1b"] = norm_spec(eps, "norm1b");
        block.parts["mixer"] = L.at("type").as_string() == "attention" ? attention_spec(L.at("mixer"), eps) : mamba2_spec(L.at("mixer"), eps);
        if (const Json* mlp = optional(L, "mlp")) {
            block.parts["norm2"] = norm_spec(eps, "norm2");
            block.parts["norm2b"] = norm_spec(eps, "norm2b");
            block.parts["feed_forward"] = mlp_spec(*mlp, spec.vocab_size);
        } else {
            for (const char* name : {"norm2", "norm2b"}) spec.ignorable.push_back(format("l%lld.%s", (long long)i, name));      // a checkpoint may carry them all the same
        }
        spec.layers.push_back(block);
    }
    // the run order: the loop's span as often as it says, a cache entry per call
    const Json* loop = optional(c, "loop");
    const int64_t a = loop ? loop->at("start").as_int() : n, b = loop ? loop->at("stop").as_int() : n, times = loop ? loop->at("times").as_int() : 0;
    auto call = [&](int64_t layer) {
        LayerCall cl;
        cl.layer = (int)layer;
        cl.cache = (int)spec.program.size();
        spec.program.push_back(cl);
    };
    for (int64_t i = 0; i < a; ++i) call(i);
    for (int64_t t = 0; t < times; ++t)
        for (int64_t i = a; i < b; ++i) call(i);
    for (int64_t i = b; i < n; ++i) call(i);
    return spec;
}

struct RegisterDapozen {
    RegisterDapozen() { register_architecture({kName, read_dapozen, dapozen_spec}); }
} register_dapozen;
}  // namespace

}  // namespace friday
