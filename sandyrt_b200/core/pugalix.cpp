// Pugalix: a decoder whose layers are windowed softmax attention, gated linear attention or a matrix memory, one each.
//
// config.json (all sizes and every constant that differs between models come from it):
//   architecture     "Pugalix"
//   vocab, width
//   embedding.scale  the factor on the embedding's rows (absent: 1)
//   norm.eps
//   layers[i]        {type: "attention" | "gla" | "mlstm", mixer: {...}, mlp: {kind: "dense", ff} | null}
//     attention      mixer {heads, kv_heads, dim, vdim, scale, rot {dims, base} | absent, mask {size, keep_first} | absent,
//                    kv_from | absent: the layer whose keys and values this one reads}
//     gla            mixer {heads, dim, vdim, tau, rank | absent: the decay's rank, which the weight file states otherwise}
//     mlstm          mixer {heads, dim, vdim, gate_cap}
//
// A layer is x += mixer(norm1(x)); x += ff(norm2(x)) with RMS norms; a layer without `mlp` is its mixer alone.  Attention
// has biases on q, k and v, rotates neighbouring pairs, adds a one to the softmax's denominator and gates its heads'
// output element by element.
// Tensors: embed, head, final.norm, and per layer l<i>.norm1 / norm2, l<i>.mix.* and l<i>.mlp.gate / up / down; linear
// weights are [out, in].
//
// The typed configuration below checks the file; `describe` turns it into parts of parts_linear.cpp and parts_hybrid.cpp.
// Nothing else in the engine knows this architecture.
#include "config.h"
#include "errors.h"

namespace sandy {

namespace {

[[noreturn]] void bad(const std::string& where, const std::string& what) { throw ConfigError("config.json: " + where + ": " + what); }

const Json* maybe(const Json& o, const std::string& key) {
    const Json* v = o.is_object() ? o.find(key) : nullptr;
    return v && !v->is_null() ? v : nullptr;
}
const Json& need(const Json& o, const std::string& where, const std::string& key) {
    const Json* v = maybe(o, key);
    if (!v) bad(where, "required key '" + key + "' is missing");
    return *v;
}
int64_t as_int(const Json& v, const std::string& where, const std::string& key) {
    if (!v.is_int()) bad(where, "'" + key + "' must be int, got " + v.dump());
    return v.as_int();
}
double as_num(const Json& v, const std::string& where, const std::string& key) {
    if (!v.is_number()) bad(where, "'" + key + "' must be a number, got " + v.dump());
    return v.as_double();
}
int64_t need_int(const Json& o, const std::string& where, const std::string& key) { return as_int(need(o, where, key), where, key); }
int64_t maybe_int(const Json& o, const std::string& where, const std::string& key, int64_t fallback) {
    const Json* v = maybe(o, key);
    return v ? as_int(*v, where, key) : fallback;
}
double need_num(const Json& o, const std::string& where, const std::string& key) { return as_num(need(o, where, key), where, key); }
const Json& as_obj(const Json& v, const std::string& where, const std::string& key) {
    if (!v.is_object()) bad(where, "'" + key + "' must be an object, got " + v.dump());
    return v;
}
void positive(int64_t v, const std::string& where, const std::string& key) {
    if (v <= 0) bad(where, "'" + key + "' must be > 0, got " + std::to_string(v));
}

}  // namespace

PugalixConfig PugalixConfig::from_json(const Json& raw) {
    if (!raw.is_object()) throw ConfigError("config.json: top level must be a JSON object");
    PugalixConfig c;
    c.vocab = need_int(raw, "top level", "vocab");
    c.width = need_int(raw, "top level", "width");
    c.norm_eps = need_num(as_obj(need(raw, "top level", "norm"), "top level", "norm"), "norm", "eps");
    if (const Json* e = maybe(raw, "embedding"))
        if (const Json* s = maybe(as_obj(*e, "top level", "embedding"), "scale")) c.embedding_scale = as_num(*s, "embedding", "scale");
    const Json& layers = need(raw, "top level", "layers");
    if (!layers.is_array() || layers.size() == 0) bad("layers", "must be a non-empty list");
    int i = 0;
    for (const Json& lj : layers.items()) {
        const std::string at = "layers[" + std::to_string(i++) + "]", ma = at + ".mixer";
        if (!lj.is_object()) bad(at, "must be an object");
        Layer l;
        const Json& type = need(lj, at, "type");
        if (!type.is_string()) bad(at, "'type' must be a string");
        l.type = type.as_string();
        const Json& m = as_obj(need(lj, at, "mixer"), at, "mixer");
        if (l.type != "attention" && l.type != "gla" && l.type != "mlstm")
            bad(at, "unknown layer type '" + l.type + "'; one of ['attention', 'gla', 'mlstm']");
        l.heads = need_int(m, ma, "heads");
        l.dim = need_int(m, ma, "dim");
        l.vdim = need_int(m, ma, "vdim");
        if (l.type == "attention") {
            l.kv_heads = maybe_int(m, ma, "kv_heads", l.heads);
            l.scale = need_num(m, ma, "scale");
            if (const Json* rot = maybe(m, "rot")) {
                as_obj(*rot, ma, "rot");
                l.rot_dims = need_int(*rot, ma + ".rot", "dims");
                l.rot_base = need_num(*rot, ma + ".rot", "base");
            }
            if (const Json* mask = maybe(m, "mask")) {
                as_obj(*mask, ma, "mask");
                l.window = maybe_int(*mask, ma + ".mask", "size", 0);
                l.keep_first = maybe_int(*mask, ma + ".mask", "keep_first", 0);
            }
            l.kv_from = maybe_int(m, ma, "kv_from", -1);
        } else if (l.type == "gla") {
            l.tau = need_num(m, ma, "tau");
            l.rank = maybe_int(m, ma, "rank", 0);
        } else {
            l.gate_cap = need_num(m, ma, "gate_cap");
        }
        if (const Json* mlp = maybe(lj, "mlp")) {
            const Json& kind = need(as_obj(*mlp, at, "mlp"), at + ".mlp", "kind");
            if (!kind.is_string() || kind.as_string() != "dense") bad(at + ".mlp", "'kind' must be 'dense', got " + kind.dump());
            l.ff = need_int(*mlp, at + ".mlp", "ff");
            positive(l.ff, at + ".mlp", "ff");
        }
        c.layers.push_back(l);
    }
    return c;
}

Json PugalixConfig::to_json() const {
    Json j = Json::object();
    j["architecture"] = kArchitecture;
    Json e = Json::object();
    e["scale"] = embedding_scale;
    j["embedding"] = e;
    Json ls = Json::array();
    for (const Layer& l : layers) {
        Json lj = Json::object(), m = Json::object();
        m["dim"] = (long long)l.dim;
        m["heads"] = (long long)l.heads;
        m["vdim"] = (long long)l.vdim;
        if (l.type == "attention") {
            m["kv_heads"] = (long long)l.kv_heads;
            if (l.kv_from >= 0) m["kv_from"] = (long long)l.kv_from;
            if (l.window) {
                Json mask = Json::object();
                mask["keep_first"] = (long long)l.keep_first;
                mask["size"] = (long long)l.window;
                m["mask"] = mask;
            }
            if (l.rot_dims) {
                Json rot = Json::object();
                rot["base"] = l.rot_base;
                rot["dims"] = (long long)l.rot_dims;
                m["rot"] = rot;
            }
            m["scale"] = l.scale;
        } else if (l.type == "gla") {
            m["tau"] = l.tau;
            if (l.rank) m["rank"] = (long long)l.rank;
        } else {
            m["gate_cap"] = l.gate_cap;
        }
        lj["mixer"] = m;
        if (l.ff) {
            Json mlp = Json::object();
            mlp["ff"] = (long long)l.ff;
            mlp["kind"] = "dense";
            lj["mlp"] = mlp;
        } else {
            lj["mlp"] = Json();
        }
        lj["type"] = l.type;
        ls.push(lj);
    }
    j["layers"] = ls;
    Json norm = Json::object();
    norm["eps"] = norm_eps;
    j["norm"] = norm;
    j["vocab"] = (long long)vocab;
    j["width"] = (long long)width;
    return j;
}

void PugalixConfig::validate() const {
    positive(vocab, "top level", "vocab");
    positive(width, "top level", "width");
    if (!(norm_eps > 0.0)) bad("norm", "'eps' must be > 0");
    for (size_t i = 0; i < layers.size(); i++) {
        const Layer& l = layers[i];
        const std::string at = "layers[" + std::to_string(i) + "]";
        positive(l.heads, at, "heads");
        positive(l.dim, at, "dim");
        positive(l.vdim, at, "vdim");
        if (l.type == "attention") {
            positive(l.kv_heads, at, "kv_heads");
            if (l.heads % l.kv_heads) bad(at, std::to_string(l.heads) + " heads do not divide into " + std::to_string(l.kv_heads) + " kv_heads");
            if (l.rot_dims < 0 || l.rot_dims > l.dim || l.rot_dims % 2) bad(at + ".rot", "'dims' must be even and at most the head's dim");
            if (l.rot_dims && !(l.rot_base > 0.0)) bad(at + ".rot", "'base' must be > 0");
            if (l.window < 0 || l.keep_first < 0) bad(at + ".mask", "'size' and 'keep_first' must not be negative");
            if (l.kv_from >= 0) {
                if (l.kv_from >= (int64_t)i) bad(at, "'kv_from' must name an earlier layer, got " + std::to_string(l.kv_from));
                const Layer& o = layers[(size_t)l.kv_from];
                if (o.type != "attention" || o.kv_from >= 0) bad(at, "'kv_from' must name an attention layer with keys and values of its own");
                if (o.kv_heads != l.kv_heads || o.dim != l.dim || o.vdim != l.vdim)
                    bad(at, "'kv_from' names a layer whose kv_heads, dim or vdim differ");
            } else if (l.kv_from != -1) {
                bad(at, "'kv_from' must name an earlier layer, got " + std::to_string(l.kv_from));
            }
        } else {
            if (l.dim > 256) bad(at, "'dim' of a recurrence is at most 256");
            if (l.type == "gla" && (!(l.tau > 0.0) || l.rank < 0 || l.rank > 512)) bad(at, "'tau' must be > 0 and 'rank' at most 512");
            if (l.type == "mlstm" && !(l.gate_cap > 0.0)) bad(at, "'gate_cap' must be > 0");
        }
    }
}

ModelSpec describe_pugalix(const PugalixConfig& cfg) {
    ModelSpec s;
    s.architecture = cfg.architecture();
    s.width = cfg.width;
    s.vocab_size = cfg.vocab;
    auto norm = [&](const std::string& name) {
        PartSpec p;
        p.kind = "rmsnorm";
        p.params["width"] = (long long)cfg.width;
        p.params["eps"] = cfg.norm_eps;
        p.tensors = {{"weight", name}};
        return p;
    };
    std::vector<int> entry;                       // the cache entry of every layer
    int entries = 0;
    for (size_t i = 0; i < cfg.layers.size(); i++) {
        const PugalixConfig::Layer& c = cfg.layers[i];
        const std::string p = "l" + std::to_string(i) + ".", x = p + "mix.";
        LayerSpec l;
        l.block = "pre_norm";
        PartSpec& m = l.mixer;
        m.params["width"] = (long long)cfg.width;
        m.params["n_heads"] = (long long)c.heads;
        m.params["qk_dim"] = (long long)c.dim;
        m.params["v_dim"] = (long long)c.vdim;
        m.tensors = {{"q", x + "q"}, {"o", x + "o"}, {"gate", x + "g"}};
        const bool reads = c.type == "attention" && c.kv_from >= 0;      // another layer's keys and values
        if (!reads) {
            m.tensors["k"] = x + "k";
            m.tensors["v"] = x + "v";
        }
        if (c.type == "attention") {
            m.kind = "windowed_attention";
            m.params["n_kv_heads"] = (long long)c.kv_heads;
            m.params["scale"] = c.scale;
            m.params["bias"] = true;
            m.params["rot_dims"] = (long long)c.rot_dims;
            if (c.rot_dims) m.params["rot_base"] = c.rot_base;
            m.params["rot_interleaved"] = true;
            m.params["window"] = c.window ? Json((long long)c.window) : Json();
            m.params["keep_first"] = (long long)c.keep_first;
            m.params["unit_sink"] = true;
            m.params["out_gate"] = true;
            m.params["own_kv"] = !reads;
            m.tensors["q_bias"] = x + "q.b";
            if (!reads) {
                m.tensors["k_bias"] = x + "k.b";
                m.tensors["v_bias"] = x + "v.b";
            }
        } else if (c.type == "gla") {
            m.kind = "gated_linear_attention";
            m.params["eps"] = cfg.norm_eps;
            m.params["tau"] = c.tau;
            m.params["rank"] = (long long)c.rank;
            m.tensors["norm"] = x + "norm";
            m.tensors["decay_in"] = x + "a1";
            m.tensors["decay_out"] = x + "a2";
            m.tensors["decay_bias"] = x + "a2.b";
        } else {
            m.kind = "matrix_memory";
            m.params["eps"] = cfg.norm_eps;
            m.params["gate_cap"] = c.gate_cap;
            m.tensors["norm"] = x + "norm";
            m.tensors["i"] = x + "i";
            m.tensors["i_bias"] = x + "i.b";
            m.tensors["f"] = x + "f";
            m.tensors["f_bias"] = x + "f.b";
        }
        l.norms["mixer"] = norm(p + "norm1");
        if (c.ff) {
            l.feed_forward.kind = "gated_mlp";
            l.feed_forward.params["width"] = (long long)cfg.width;
            l.feed_forward.params["inner"] = (long long)c.ff;
            l.feed_forward.params["activation"] = "silu";
            l.feed_forward.tensors = {{"gate", p + "mlp.gate"}, {"up", p + "mlp.up"}, {"down", p + "mlp.down"}};
            l.norms["feed_forward"] = norm(p + "norm2");
        } else {
            l.feed_forward.kind = "none";
        }
        s.layers.push_back(std::move(l));
        LayerCall call;
        call.layer = (int)i;
        call.cache = reads ? entry[(size_t)c.kv_from] : entries++;
        call.write_cache = !reads;
        entry.push_back(call.cache);
        s.schedule.push_back(call);
    }
    s.embedding.kind = "token_embedding";
    s.embedding.params["vocab_size"] = (long long)cfg.vocab;
    s.embedding.params["width"] = (long long)cfg.width;
    s.embedding.params["scale"] = cfg.embedding_scale;
    s.embedding.tensors = {{"weight", "embed"}};
    s.position.kind = "none";
    s.final_norm = norm("final.norm");
    s.head.kind = "output_head";
    s.head.params["vocab_size"] = (long long)cfg.vocab;
    s.head.params["width"] = (long long)cfg.width;
    s.head.params["tied"] = false;
    s.head.tensors = {{"weight", "head"}};
    return s;
}

}  // namespace sandy
