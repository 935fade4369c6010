#include "stack_config.h"

#include <initializer_list>

#include "json.h"

namespace l2b {

namespace {

struct ConfigError {
    std::string what;
};

const JsonValue& need(const JsonValue& o, const char* key, const std::string& where) {
    const JsonValue* v = o.find(key);
    if (!v || v->is_null()) throw ConfigError{where + "." + key + " is missing"};
    return *v;
}
double number(const JsonValue& o, const char* key, const std::string& where) {
    const JsonValue& v = need(o, key, where);
    if (v.kind != JsonValue::NUMBER) throw ConfigError{where + "." + key + " must be a number"};
    return v.num;
}
int integer(const JsonValue& o, const char* key, const std::string& where, int lo) {
    const double d = number(o, key, where);
    if (d != (double)(int64_t)d || d < lo || d > 2147483647.0) throw ConfigError{where + "." + key + " must be an integer of at least " + std::to_string(lo)};
    return (int)d;
}

// ---- mixers ------------------------------------------------------------------------------------
void parse_latent_attention(const JsonValue& m, MixerConfig& c, const std::string& where) {
    c.kind = MixerKind::LatentAttention;
    c.heads = integer(m, "heads", where, 1);
    c.dim = integer(m, "dim", where, 1);
    c.rot_dim = integer(m, "rot_dim", where, 2);
    c.vdim = integer(m, "vdim", where, 1);
    c.kv_rank = integer(m, "kv_rank", where, 1);
    c.scale = (float)number(m, "scale", where);
    const JsonValue& r = need(m, "rot", where);
    c.rot.base = number(r, "base", where + ".rot");
    c.rot.dims = integer(r, "dims", where + ".rot", 2);
    if (c.rot.dims > c.rot_dim || c.rot.dims % 2 || c.rot_dim % 2 || !(c.rot.base > 0)) throw ConfigError{where + ".rot does not fit rot_dim"};
}

// Two softmax maps per head over the same values, the second subtracted with a learned weight; keys and values per group of heads,
// grouped by chunks of positions, or taken from another layer.
void parse_differential_attention(const JsonValue& m, MixerConfig& c, const std::string& where) {
    c.kind = MixerKind::DifferentialAttention;
    c.heads = integer(m, "heads", where, 1);
    c.kv_heads = integer(m, "kv_heads", where, 1);
    c.dim = integer(m, "dim", where, 1);
    c.vdim = integer(m, "vdim", where, 1);
    c.scale = (float)number(m, "scale", where);
    c.diff = (float)number(m, "diff", where);
    if (c.heads % c.kv_heads) throw ConfigError{where + ".heads must be a multiple of kv_heads"};
    const JsonValue* mask = m.find("mask");
    if (mask && !mask->is_null()) c.chunk = integer(*mask, "size", where + ".mask", 1);
    const JsonValue* r = m.find("rot");
    if (r && !r->is_null()) {
        c.rot.base = number(*r, "base", where + ".rot");
        c.rot.dims = integer(*r, "dims", where + ".rot", 2);
        if (c.rot.dims > c.dim || c.rot.dims % 2 || !(c.rot.base > 0)) throw ConfigError{where + ".rot does not fit dim"};
    }
    const JsonValue* from = m.find("kv_from");
    if (from && !from->is_null()) c.kv_from = integer(m, "kv_from", where, 0);
}

void parse_mlstm(const JsonValue& m, MixerConfig& c, const std::string& where) {
    c.kind = MixerKind::Mlstm;
    c.heads = integer(m, "heads", where, 1);
    c.dim = integer(m, "dim", where, 1);
    c.vdim = integer(m, "vdim", where, 1);
    c.gate_cap = (float)number(m, "gate_cap", where);
    if (!(c.gate_cap > 0.f)) throw ConfigError{where + ".gate_cap must be positive"};
}

struct MixerEntry {
    const char* type;
    void (*parse)(const JsonValue&, MixerConfig&, const std::string&);
};
const MixerEntry kLatent = {"latent_attention", parse_latent_attention};
const MixerEntry kDifferential = {"attention", parse_differential_attention};
const MixerEntry kMlstm = {"mlstm", parse_mlstm};

// ---- designs -----------------------------------------------------------------------------------
// The list of layers; a design names the mixers its layers may have and its feed-forward.
void parse_layers(const JsonValue& root, StackConfig& c, std::initializer_list<const MixerEntry*> mixers, MlpKind dense) {
    const JsonValue& ls = need(root, "layers", "config");
    if (ls.kind != JsonValue::ARRAY || ls.items.empty()) throw ConfigError{"config.layers must be a list of layers"};
    for (size_t i = 0; i < ls.items.size(); ++i) {
        const JsonValue& l = ls.items[i];
        const std::string where = "config.layers[" + std::to_string(i) + "]";
        const JsonValue& type = need(l, "type", where);
        StackLayerConfig out;
        const MixerEntry* found = nullptr;
        for (const MixerEntry* e : mixers)
            if (type.kind == JsonValue::STRING && type.str == e->type) found = e;
        if (!found) throw ConfigError{where + ": unknown mixer type '" + type.str + "'"};
        found->parse(need(l, "mixer", where), out.mix, where + ".mixer");
        const JsonValue* mlp = l.find("mlp");
        if (mlp && !mlp->is_null()) {
            const JsonValue& kind = need(*mlp, "kind", where + ".mlp");
            if (kind.str != "dense") throw ConfigError{where + ": unknown feed-forward kind '" + kind.str + "'"};
            out.mlp = dense;
            out.ff = integer(*mlp, "ff", where + ".mlp", 1);
        }
        if (const int j = out.mix.kv_from; j >= 0) {
            if (j >= (int)i) throw ConfigError{where + ".mixer.kv_from must name an earlier layer"};
            const MixerConfig& own = c.layers[j].mix;
            if (own.kind != out.mix.kind || own.kv_from >= 0) throw ConfigError{where + ".mixer.kv_from names a layer without keys and values of its own"};
            if (own.kv_heads != out.mix.kv_heads || own.dim != out.mix.dim || own.vdim != out.mix.vdim)
                throw ConfigError{where + ".mixer does not fit the keys and values of layer " + std::to_string(j) + " (kv_from)"};
        }
        c.layers.push_back(out);
    }
}

// Savozen: latent attention (one cached latent and one shared rotated key per position, a sink in the softmax, an output gate),
// dynamic-tanh norms, a gated feed-forward with tanh-gelu, a per-layer token input, and a stretch of layers that is run several
// times with a step vector added before each pass.
void parse_savozen(const JsonValue& root, StackConfig& c) {
    c.norm = NormKind::DynamicTanh;
    c.vocab = integer(root, "vocab", "config", 1);
    c.width = integer(root, "width", "config", 1);
    if (const JsonValue* e = root.find("embedding"))
        if (!e->is_null()) c.embed_scale = (float)number(*e, "scale", "config.embedding");
    c.eps = (float)number(need(root, "norm", "config"), "eps", "config.norm");
    parse_layers(root, c, {&kLatent}, MlpKind::GatedGeluTanh);
    const JsonValue* loop = root.find("loop");
    if (loop && !loop->is_null()) {
        c.loop_start = integer(*loop, "start", "config.loop", 0);
        c.loop_stop = integer(*loop, "stop", "config.loop", 0);
        c.loop_times = integer(*loop, "times", "config.loop", 1);
        if (c.loop_stop <= c.loop_start || c.loop_stop > (int)c.layers.size()) throw ConfigError{"config.loop does not name a range of layers"};
    }
    const JsonValue* side = root.find("token_side");
    if (side && !side->is_null()) c.side_dim = integer(*side, "dim", "config.token_side", 1);
}

// Perezen: differential attention within chunks of positions (some layers on another layer's keys and values) and matrix-memory
// recurrences (mLSTM), learned position vectors, rms norms before and after every sublayer, a gated feed-forward with silu.
void parse_perezen(const JsonValue& root, StackConfig& c) {
    c.norm = NormKind::Rms;
    c.post_norm = true;
    c.vocab = integer(root, "vocab", "config", 1);
    c.width = integer(root, "width", "config", 1);
    c.max_positions = integer(root, "max_positions", "config", 1);
    c.logit_scale = (float)number(root, "logit_scale", "config");
    c.eps = (float)number(need(root, "norm", "config"), "eps", "config.norm");
    parse_layers(root, c, {&kDifferential, &kMlstm}, MlpKind::GatedSilu);
}

struct DesignEntry {
    const char* architecture;
    void (*parse)(const JsonValue&, StackConfig&);
};
const DesignEntry kDesigns[] = {
    {"Savozen", parse_savozen},
    {"Perezen", parse_perezen},
};

}  // namespace

bool StackConfig::recurrent() const {
    for (const StackLayerConfig& l : layers)
        if (l.mix.kind == MixerKind::Mlstm) return true;
    return false;
}

std::vector<LayerRun> StackConfig::runs() const {
    std::vector<LayerRun> r;
    const int n = (int)layers.size();
    if (!has_loop()) {
        for (int i = 0; i < n; ++i) r.push_back({i, -1});
        return r;
    }
    for (int i = 0; i < loop_start; ++i) r.push_back({i, -1});
    for (int t = 0; t < loop_times; ++t)
        for (int i = loop_start; i < loop_stop; ++i) r.push_back({i, i == loop_start ? t : -1});
    for (int i = loop_stop; i < n; ++i) r.push_back({i, -1});
    return r;
}

bool parse_stack_config(const char* json, size_t n, StackConfig& out, std::string& err) {
    JsonValue root;
    if (!JsonParser::parse(json, n, root) || root.kind != JsonValue::OBJECT) {
        err = "the model configuration is not a JSON object";
        return false;
    }
    const JsonValue* a = root.find("architecture");
    const std::string arch = a ? a->str : "";
    for (const DesignEntry& d : kDesigns)
        if (arch == d.architecture) {
            try {
                out = StackConfig();
                out.architecture = arch;
                d.parse(root, out);
                return true;
            } catch (const ConfigError& e) {
                err = e.what;
                return false;
            }
        }
    err = "unsupported model architecture: " + arch;
    return false;
}

}  // namespace l2b
