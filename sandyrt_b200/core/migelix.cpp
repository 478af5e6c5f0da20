// Migelix: a decoder whose layers are time mixing, windowed softmax attention, or attention beside a delta rule.
//
// config.json (all sizes and every constant that differs between models come from it):
//   architecture     "Migelix"
//   vocab, width
//   norm.eps
//   logit_softcap    the cap of the logits (absent: none)
//   layers[i]        {type: "wkv" | "attention" | "parallel", mixer: {...}, mlp: {kind: "dense", ff} | null,
//                    weights_of | absent: the layer whose tensors this one uses, with a cache or state of its own}
//     attention      mixer {heads, kv_heads, dim, vdim, scale, softcap | absent, rot | absent, mask {size} | absent}
//                    rot {dims, base, scaling {factor, original, fast, slow} | absent}
//     parallel       mixer {left: {as attention, no softcap}, right: {heads, kv_heads, dim, vdim, conv}, left_scale, right_scale}
//     wkv            mixer {heads, dim}
//   The ranks of the low-rank products are the weight file's; a configuration may state them (`rank` in wkv and right,
//   `gate_rank` in right), which only matters where weights are drawn at random.
//
// A layer is x += mixer(norm1(x)); x += ff(norm2(x)) with RMS norms whose weights are stored around zero; a layer without `mlp`
// is its mixer alone.  Both attentions take the keys as projected for their values and rotate neighbouring pairs.  The single
// one caps its scores and gates its heads element by element; the one beside the delta rule has biases on q and k and a learned
// sink.  The head reads the embedding's table.
// Tensors: embed, final.norm, and per layer with tensors of its own l<i>.norm1 / norm2, l<i>.mix.* (a parallel mixer's under
// .left and .right) and l<i>.mlp.gate / up / down; linear weights are [out, in].
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
double maybe_num(const Json& o, const std::string& where, const std::string& key, double fallback) {
    const Json* v = maybe(o, key);
    return v ? as_num(*v, where, key) : fallback;
}
const Json& as_obj(const Json& v, const std::string& where, const std::string& key) {
    if (!v.is_object()) bad(where, "'" + key + "' must be an object, got " + v.dump());
    return v;
}
void positive(int64_t v, const std::string& where, const std::string& key) {
    if (v <= 0) bad(where, "'" + key + "' must be > 0, got " + std::to_string(v));
}

MigelixConfig::Attention read_attention(const Json& m, const std::string& at) {
    MigelixConfig::Attention a;
    a.heads = need_int(m, at, "heads");
    a.kv_heads = maybe_int(m, at, "kv_heads", a.heads);
    a.dim = need_int(m, at, "dim");
    a.vdim = maybe_int(m, at, "vdim", a.dim);
    a.scale = need_num(m, at, "scale");
    a.softcap = maybe_num(m, at, "softcap", 0.0);
    if (const Json* mask = maybe(m, "mask")) a.window = maybe_int(as_obj(*mask, at, "mask"), at + ".mask", "size", 0);
    if (const Json* rot = maybe(m, "rot")) {
        as_obj(*rot, at, "rot");
        a.rot_dims = need_int(*rot, at + ".rot", "dims");
        a.rot_base = need_num(*rot, at + ".rot", "base");
        if (const Json* s = maybe(*rot, "scaling")) {
            const std::string sa = at + ".rot.scaling";
            as_obj(*s, at + ".rot", "scaling");
            a.yarn = true;
            a.yarn_factor = need_num(*s, sa, "factor");
            a.yarn_original = need_num(*s, sa, "original");
            a.yarn_fast = need_num(*s, sa, "fast");
            a.yarn_slow = need_num(*s, sa, "slow");
        }
    }
    return a;
}

Json attention_json(const MigelixConfig::Attention& a) {
    Json m = Json::object();
    m["dim"] = (long long)a.dim;
    m["heads"] = (long long)a.heads;
    m["kv_heads"] = (long long)a.kv_heads;
    if (a.window) {
        Json mask = Json::object();
        mask["size"] = (long long)a.window;
        m["mask"] = mask;
    }
    if (a.rot_dims) {
        Json rot = Json::object();
        rot["base"] = a.rot_base;
        rot["dims"] = (long long)a.rot_dims;
        if (a.yarn) {
            Json s = Json::object();
            s["factor"] = a.yarn_factor;
            s["fast"] = a.yarn_fast;
            s["original"] = a.yarn_original;
            s["slow"] = a.yarn_slow;
            rot["scaling"] = s;
        }
        m["rot"] = rot;
    }
    m["scale"] = a.scale;
    if (a.softcap != 0.0) m["softcap"] = a.softcap;
    m["vdim"] = (long long)a.vdim;
    return m;
}

void check_attention(const MigelixConfig::Attention& a, const std::string& at) {
    positive(a.heads, at, "heads");
    positive(a.kv_heads, at, "kv_heads");
    positive(a.dim, at, "dim");
    if (a.heads % a.kv_heads) bad(at, std::to_string(a.heads) + " heads do not divide into " + std::to_string(a.kv_heads) + " kv_heads");
    if (a.vdim != a.dim) bad(at, "the values are the keys: 'vdim' must be 'dim'");
    if (a.softcap < 0.0) bad(at, "'softcap' must not be negative");
    if (a.window < 0) bad(at + ".mask", "'size' must not be negative");
    if (a.rot_dims < 0 || a.rot_dims > a.dim || a.rot_dims % 2) bad(at + ".rot", "'dims' must be even and at most the head's dim");
    if (a.rot_dims && !(a.rot_base > 0.0)) bad(at + ".rot", "'base' must be > 0");
    if (a.yarn && (!(a.yarn_factor > 0.0) || !(a.yarn_original > 0.0) || !(a.yarn_fast > 0.0) || !(a.yarn_slow > 0.0) || a.rot_base == 1.0))
        bad(at + ".rot.scaling", "'factor', 'original', 'fast' and 'slow' must be > 0, and the base not 1");
}

}  // namespace

MigelixConfig MigelixConfig::from_json(const Json& raw) {
    if (!raw.is_object()) throw ConfigError("config.json: top level must be a JSON object");
    MigelixConfig c;
    c.vocab = need_int(raw, "top level", "vocab");
    c.width = need_int(raw, "top level", "width");
    c.norm_eps = need_num(as_obj(need(raw, "top level", "norm"), "top level", "norm"), "norm", "eps");
    c.logit_softcap = maybe_num(raw, "top level", "logit_softcap", 0.0);
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
        if (l.type != "attention" && l.type != "parallel" && l.type != "wkv")
            bad(at, "unknown layer type '" + l.type + "'; one of ['attention', 'parallel', 'wkv']");
        const Json& m = as_obj(need(lj, at, "mixer"), at, "mixer");
        if (l.type == "attention") {
            l.attention = read_attention(m, ma);
        } else if (l.type == "parallel") {
            l.attention = read_attention(as_obj(need(m, ma, "left"), ma, "left"), ma + ".left");
            const Json& r = as_obj(need(m, ma, "right"), ma, "right");
            const std::string ra = ma + ".right";
            l.left_scale = need_num(m, ma, "left_scale");
            l.right_scale = need_num(m, ma, "right_scale");
            l.heads = need_int(r, ra, "heads");
            l.kv_heads = maybe_int(r, ra, "kv_heads", l.heads);
            l.dim = need_int(r, ra, "dim");
            l.vdim = need_int(r, ra, "vdim");
            l.conv = need_int(r, ra, "conv");
            l.rank = maybe_int(r, ra, "rank", 0);
            l.gate_rank = maybe_int(r, ra, "gate_rank", 0);
        } else {
            l.heads = need_int(m, ma, "heads");
            l.dim = need_int(m, ma, "dim");
            l.rank = maybe_int(m, ma, "rank", 0);
        }
        if (const Json* mlp = maybe(lj, "mlp")) {
            const Json& kind = need(as_obj(*mlp, at, "mlp"), at + ".mlp", "kind");
            if (!kind.is_string() || kind.as_string() != "dense") bad(at + ".mlp", "'kind' must be 'dense', got " + kind.dump());
            l.ff = need_int(*mlp, at + ".mlp", "ff");
            positive(l.ff, at + ".mlp", "ff");
        }
        l.weights_of = maybe_int(lj, at, "weights_of", -1);
        if (maybe(lj, "weights_of") && l.weights_of < 0) bad(at, "'weights_of' must name a layer, got " + std::to_string(l.weights_of));
        c.layers.push_back(l);
    }
    return c;
}

Json MigelixConfig::layer_json(const Layer& l) {
    Json lj = Json::object(), m = Json::object();
    if (l.type == "attention") {
        m = attention_json(l.attention);
    } else if (l.type == "parallel") {
        m["left"] = attention_json(l.attention);
        m["left_scale"] = l.left_scale;
        Json r = Json::object();
        r["conv"] = (long long)l.conv;
        r["dim"] = (long long)l.dim;
        if (l.gate_rank) r["gate_rank"] = (long long)l.gate_rank;
        r["heads"] = (long long)l.heads;
        r["kv_heads"] = (long long)l.kv_heads;
        if (l.rank) r["rank"] = (long long)l.rank;
        r["vdim"] = (long long)l.vdim;
        m["right"] = r;
        m["right_scale"] = l.right_scale;
    } else {
        m["dim"] = (long long)l.dim;
        m["heads"] = (long long)l.heads;
        if (l.rank) m["rank"] = (long long)l.rank;
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
    return lj;
}

Json MigelixConfig::to_json() const {
    Json j = Json::object();
    j["architecture"] = kArchitecture;
    Json ls = Json::array();
    for (const Layer& l : layers) {
        Json lj = layer_json(l);
        if (l.weights_of >= 0) lj["weights_of"] = (long long)l.weights_of;
        ls.push(lj);
    }
    j["layers"] = ls;
    if (logit_softcap != 0.0) j["logit_softcap"] = logit_softcap;
    Json norm = Json::object();
    norm["eps"] = norm_eps;
    j["norm"] = norm;
    j["vocab"] = (long long)vocab;
    j["width"] = (long long)width;
    return j;
}

void MigelixConfig::validate() const {
    positive(vocab, "top level", "vocab");
    positive(width, "top level", "width");
    if (!(norm_eps > 0.0)) bad("norm", "'eps' must be > 0");
    if (logit_softcap < 0.0) bad("top level", "'logit_softcap' must not be negative");
    for (size_t i = 0; i < layers.size(); i++) {
        const Layer& l = layers[i];
        const std::string at = "layers[" + std::to_string(i) + "]";
        if (l.type != "wkv") check_attention(l.attention, l.type == "attention" ? at + ".mixer" : at + ".mixer.left");
        if (l.type == "parallel") {
            const std::string ra = at + ".mixer.right";
            positive(l.heads, ra, "heads");
            positive(l.kv_heads, ra, "kv_heads");
            positive(l.dim, ra, "dim");
            positive(l.vdim, ra, "vdim");
            if (l.heads % l.kv_heads) bad(ra, std::to_string(l.heads) + " heads do not divide into " + std::to_string(l.kv_heads) + " kv_heads");
            if (l.dim > 256) bad(ra, "'dim' of a recurrence is at most 256");
            if (l.conv < 1 || l.conv > 8) bad(ra, "'conv' must be 1 .. 8 taps, got " + std::to_string(l.conv));
            if (l.rank < 0 || l.rank > 512 || l.gate_rank < 0 || l.gate_rank > 512) bad(ra, "ranks are at most 512");
        }
        if (l.type == "wkv") {
            positive(l.heads, at + ".mixer", "heads");
            positive(l.dim, at + ".mixer", "dim");
            if (l.dim > 256) bad(at + ".mixer", "'dim' of a recurrence is at most 256");
            if (l.rank < 0 || l.rank > 512) bad(at + ".mixer", "'rank' is at most 512");
        }
        if (l.weights_of >= 0) {
            const size_t j = owner(i);
            if (layer_json(layers[j]).dump() != layer_json(l).dump())
                bad(at, "uses the tensors of layer " + std::to_string(j) + ", whose sizes or constants differ");
        }
    }
}

// The layer whose tensors layer i uses.
size_t MigelixConfig::owner(size_t i) const {
    size_t at = i;
    for (size_t hops = 0; layers[at].weights_of >= 0; hops++) {
        if ((size_t)layers[at].weights_of >= layers.size() || hops >= layers.size())
            bad("layers[" + std::to_string(i) + "]", "'weights_of' must lead to a layer with tensors of its own");
        at = (size_t)layers[at].weights_of;
    }
    return at;
}

ModelSpec describe_migelix(const MigelixConfig& cfg) {
    ModelSpec s;
    s.architecture = cfg.architecture();
    s.width = cfg.width;
    s.vocab_size = cfg.vocab;
    auto norm = [&](const std::string& name) {
        PartSpec p;
        p.kind = "rmsnorm";
        p.params["width"] = (long long)cfg.width;
        p.params["eps"] = cfg.norm_eps;
        p.params["gain_offset"] = 1.0;
        p.tensors = {{"weight", name}};
        return p;
    };
    // `pre`: in front of the part's parameter and tensor names, `x` in front of the weight file's
    auto attention = [&](PartSpec& m, const MigelixConfig::Attention& a, const std::string& pre, const std::string& x) {
        m.params[pre + "n_heads"] = (long long)a.heads;
        m.params[pre + "n_kv_heads"] = (long long)a.kv_heads;
        m.params[pre + "qk_dim"] = (long long)a.dim;
        m.params[pre + "v_dim"] = (long long)a.vdim;
        m.params[pre + "scale"] = a.scale;
        m.params[pre + "values_are_keys"] = true;
        m.params[pre + "rot_dims"] = (long long)a.rot_dims;
        if (a.rot_dims) m.params[pre + "rot_base"] = a.rot_base;
        m.params[pre + "rot_interleaved"] = true;
        if (a.yarn) {
            Json y = Json::object();
            y["factor"] = a.yarn_factor;
            y["original"] = a.yarn_original;
            y["fast"] = a.yarn_fast;
            y["slow"] = a.yarn_slow;
            m.params[pre + "rot_yarn"] = y;
        }
        m.params[pre + "window"] = a.window ? Json((long long)a.window) : Json();
        m.params[pre + "softcap"] = a.softcap;
        for (const char* n : {"q", "k", "o"}) m.tensors[pre + n] = x + n;
    };
    std::map<size_t, int> built;                  // layer of the configuration -> layer of the description
    for (size_t i = 0; i < cfg.layers.size(); i++) {
        if (cfg.layers[i].weights_of >= 0) continue;
        const MigelixConfig::Layer& c = cfg.layers[i];
        const std::string p = "l" + std::to_string(i) + ".", x = p + "mix.";
        LayerSpec l;
        l.block = "pre_norm";
        PartSpec& m = l.mixer;
        m.params["width"] = (long long)cfg.width;
        if (c.type == "attention") {
            m.kind = "windowed_attention";
            attention(m, c.attention, "", x);
            m.params["out_gate"] = true;
            m.tensors["gate"] = x + "g";
        } else if (c.type == "parallel") {
            m.kind = "attention_beside_channel_delta";
            m.params["eps"] = cfg.norm_eps;
            m.params["left_scale"] = c.left_scale;
            m.params["right_scale"] = c.right_scale;
            attention(m, c.attention, "left.", x + "left.");
            m.params["left.bias"] = true;
            m.params["left.sink"] = true;
            m.tensors["left.q_bias"] = x + "left.q.b";
            m.tensors["left.k_bias"] = x + "left.k.b";
            m.tensors["left.sink"] = x + "left.sink";
            m.params["right.n_heads"] = (long long)c.heads;
            m.params["right.n_qk_heads"] = (long long)c.kv_heads;
            m.params["right.qk_dim"] = (long long)c.dim;
            m.params["right.v_dim"] = (long long)c.vdim;
            m.params["right.conv_taps"] = (long long)c.conv;
            m.params["right.rank"] = (long long)c.rank;
            m.params["right.gate_rank"] = (long long)c.gate_rank;
            const std::map<std::string, std::string> names = {
                {"q", "q"}, {"k", "k"}, {"v", "v"}, {"o", "o"}, {"norm", "norm"}, {"q_conv", "q.conv"}, {"k_conv", "k.conv"}, {"v_conv", "v.conv"},
                {"beta", "b"}, {"decay_in", "a1"}, {"decay_out", "a2"}, {"dt_bias", "dt_bias"}, {"a_log", "A_log"}, {"gate_in", "g1"}, {"gate_out", "g2"}};
            for (const auto& n : names) m.tensors["right." + n.first] = x + "right." + n.second;
        } else {
            m.kind = "time_mixing";
            m.params["eps"] = cfg.norm_eps;
            m.params["n_heads"] = (long long)c.heads;
            m.params["dim"] = (long long)c.dim;
            m.params["rank"] = (long long)c.rank;
            m.tensors = {{"r", x + "r"}, {"k", x + "k"}, {"v", x + "v"}, {"gate", x + "g"}, {"decay_in", x + "w1"}, {"decay_out", x + "w2"},
                         {"decay_bias", x + "w0"}, {"bonus", x + "u"}, {"norm", x + "norm"}, {"o", x + "o"}};
            for (const char* n : {"r", "k", "v", "g", "w"}) m.tensors[std::string("mu_") + n] = x + "mu." + n;
        }
        l.norms["mixer"] = norm(p + "norm1");
        if (c.ff) {
            l.feed_forward.kind = "gated_mlp";
            l.feed_forward.params["width"] = (long long)cfg.width;
            l.feed_forward.params["inner"] = (long long)c.ff;
            l.feed_forward.params["activation"] = "gelu_tanh";
            l.feed_forward.tensors = {{"gate", p + "mlp.gate"}, {"up", p + "mlp.up"}, {"down", p + "mlp.down"}};
            l.norms["feed_forward"] = norm(p + "norm2");
        } else {
            l.feed_forward.kind = "none";
        }
        built[i] = (int)s.layers.size();
        s.layers.push_back(std::move(l));
    }
    for (size_t i = 0; i < cfg.layers.size(); i++) {
        LayerCall call;
        call.layer = built.at(cfg.owner(i));
        call.cache = (int)i;
        s.schedule.push_back(call);
    }
    s.embedding.kind = "token_embedding";
    s.embedding.params["vocab_size"] = (long long)cfg.vocab;
    s.embedding.params["width"] = (long long)cfg.width;
    s.embedding.tensors = {{"weight", "embed"}};
    s.position.kind = "none";
    s.final_norm = norm("final.norm");
    s.head.kind = "output_head";
    s.head.params["vocab_size"] = (long long)cfg.vocab;
    s.head.params["width"] = (long long)cfg.width;
    s.head.params["tied"] = true;
    if (cfg.logit_softcap != 0.0) s.head.params["logit_softcap"] = cfg.logit_softcap;
    return s;
}

}  // namespace sandy
