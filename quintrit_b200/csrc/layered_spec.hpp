// Description of a decoder whose layers differ from one another, and the registry that turns a model folder (config.json +
// model.safetensors) into one. A layer is a token mixer - a recurrence or an attention, or two of them side by side - and a feed-forward,
// each with its own sizes and constants; a design is an entry of kLayeredDesigns: it names its config keys and tensors and fills the description.
#pragma once
#include <cstdint>
#include <cstdio>
#include <fstream>
#include <functional>
#include <sstream>
#include <string>
#include <vector>

#include "capi_common.cuh"
#include "json.hpp"
#include "safetensors.hpp"

namespace qtb {

enum class MixerKind { kMamba2, kHgrn2, kAttention, kRetention, kLogistic };

inline const char* mixer_name(MixerKind k) {
    switch (k) {
        case MixerKind::kMamba2: return "mamba2";
        case MixerKind::kHgrn2: return "hgrn2";
        case MixerKind::kAttention: return "attention";
        case MixerKind::kRetention: return "retention";
        default: return "logistic_attention";
    }
}

struct MixerSpec {
    MixerKind kind = MixerKind::kAttention;
    int heads = 0;
    int dim = 0, vdim = 0;                // query / key size (all but mamba2) and value size of a head
    int state = 0, groups = 0;            // mamba2: state size, groups that share B and C
    int conv = 0, norm_groups = 0;        // mamba2: taps of the short convolution, parts of the output norm
    int kv_heads = 0;                     // attentions
    float scale = 1.0f;                   // attentions: factor of q . k
    int window = 0;                       // attention: position i sees j with 0 <= i - j < window
    int pool = 0;                         // attention: block size of the pooled keys and values before the window, 0 = none
    bool head_gate = false;               // attention: one sigmoid per head on the output
    std::vector<float> decay;             // retention: one factor per head
    int rot_dims = 0;                     // retention: rotated dimensions of a head, 0 = none
    double rot_base = 1.0;
    float temp_coef = 0.0f, temp_every = 1.0f;  // logistic attention: q times 1 + coef ln(floor((p + 1) / every) + 1)
    bool value_norm = false;              // logistic attention: values divided by their root mean square
    bool distance_bias = false;           // logistic attention: slope_h (i - j) is taken off a score
    // tensor names
    std::vector<std::string> in;          // projections, stacked row-wise in the order the mixer kernels read them
    std::string out;
    std::string conv_w, conv_b, dt_bias, a_log, d_skip, mix_norm, f_bias, lower, q_norm, k_norm, logit_bias;
    std::string result_norm;              // norm of W_o's result over the model width, empty: none

    int inner() const { return heads * vdim; }                          // width of the mixer's output before the output projection
    int conv_dim() const { return inner() + 2 * groups * state; }       // mamba2: channels of the convolution (x | B | C)
    int key_dim() const { return kind == MixerKind::kMamba2 ? state : dim; }  // rows of a head's recurrent state
    bool cached() const { return kind == MixerKind::kAttention || kind == MixerKind::kLogistic; }  // keys and values, not a recurrent state
    int in_rows() const {
        switch (kind) {
            case MixerKind::kMamba2: return 2 * inner() + 2 * groups * state + heads;                             // z | x | B | C | dt
            case MixerKind::kHgrn2: return 2 * heads * dim + inner();                                             // q | f | v
            case MixerKind::kRetention: return 2 * heads * dim + 2 * inner();                                     // q | k | v | g
            case MixerKind::kLogistic: return heads * dim + kv_heads * (dim + vdim);                              // q | k | v
            default: return heads * dim + kv_heads * (dim + vdim) + (head_gate ? heads : 0);                      // q | k | v | g
        }
    }
    int gate_col() const { return 2 * heads * dim + inner(); }          // retention: first projection row of g
};

enum class FfKind { kNone, kDense, kExperts };

struct LayerSpec {
    std::vector<MixerSpec> mixers;        // one, or two side by side whose normed results are averaged
    // parallel: x + mixer(norm1 x) + ff(norm2 x); else x' = x + mixer(norm1 x), then x' + ff(norm2 x')
    bool parallel = false;
    bool gated_residual = false;          // parallel: each sublayer's result is multiplied by sigmoid(W h + b) before it is added
    FfKind ff_kind = FfKind::kNone;
    int ff = 0;                           // feed-forward width (SwiGLU); of one expert where there are several
    int experts = 0, top = 0;             // experts: their number, how many a token uses
    int expert_groups = 1, keep_groups = 1;  // neighbours form groups; only those of the best groups can be chosen
    float router_scale = 1.0f;
    int shared_ff = 0;                    // experts: width of the expert that every token uses, times sigmoid(w h)
    // tensor names
    std::string norm1, norm2, gate1, gate1_bias, gate2, gate2_bias, ff_gate, ff_up, ff_down;
    std::string expert_prefix, router, shared_gate, shared_up, shared_down, shared_scale;  // expert e: prefix + e + ".gate" / ".up" / ".down"
    std::string depth;                    // weights of the averages over the embedding output and the layers' results, empty: none

    int in_rows() const {
        int n = 0;
        for (const MixerSpec& m : mixers) n += m.in_rows();
        return n;
    }
};

enum class NormKind { kRms, kTanh };  // RMS norm; tanh(alpha x) w + b

struct LayeredSpec {
    std::string design;
    int width = 0, vocab = 0, max_positions = 0;  // max_positions 0: no bound of the model's own
    float eps = 0.0f, embed_scale = 1.0f;
    NormKind norm = NormKind::kRms;       // the layers' norms and the final one
    std::vector<LayerSpec> layers;
    std::string embed, pos, head, embed_norm, out_norm;  // pos empty: no position vectors; head: the output table (the embedding when tied); embed_norm empty: none
};

// ---- config.json ------------------------------------------------------------------------------------------------------------------
// Reads required keys; the first failure is remembered and the rest give neutral values, so that a reader checks once at the end.
struct ConfigReader {
    std::string error;
    void fail_key(const std::string& where, const char* key, const char* what) {
        if (error.empty()) error = "config.json: " + where + key + " " + what;
    }
    const JsonValue* object(const JsonValue& v, const std::string& where, const char* key) {
        static const JsonValue empty;
        const JsonValue* p = v.get(key);
        if (p == nullptr || !p->is(JsonValue::kObject)) {
            fail_key(where, key, "is missing or not an object");
            return &empty;
        }
        return p;
    }
    // An object that may be left out (or null).
    const JsonValue* optional(const JsonValue& v, const std::string& where, const char* key) {
        const JsonValue* p = v.get(key);
        return p == nullptr || p->is(JsonValue::kNull) ? nullptr : object(v, where, key);
    }
    int size(const JsonValue& v, const std::string& where, const char* key) {
        const JsonValue* p = v.get(key);
        uint64_t u = 0;
        if (p == nullptr || !p->as_u64(&u) || u == 0 || u > (1u << 28)) {
            fail_key(where, key, "is missing or not a positive integer");
            return 1;
        }
        return static_cast<int>(u);
    }
    float number(const JsonValue& v, const std::string& where, const char* key) {
        const JsonValue* p = v.get(key);
        if (p == nullptr || !p->is(JsonValue::kNumber)) {
            fail_key(where, key, "is missing or not a number");
            return 1.0f;
        }
        return static_cast<float>(p->number());
    }
    double real(const JsonValue& v, const std::string& where, const char* key) {
        number(v, where, key);
        const JsonValue* p = v.get(key);
        return p != nullptr && p->is(JsonValue::kNumber) ? p->number() : 1.0;
    }
    std::string text(const JsonValue& v, const std::string& where, const char* key) {
        const JsonValue* p = v.get(key);
        if (p == nullptr || !p->is(JsonValue::kString)) {
            fail_key(where, key, "is missing or not a string");
            return "";
        }
        return p->s;
    }
};

// Lasosun: parallel layers with two norms and gated residuals; mixers mamba2, hgrn2 and attention (sliding window with pooled blocks, one
// output gate per head, no rotation); learned positions; tied embedding.
inline std::string read_lasosun(const JsonValue& cfg, LayeredSpec* out) {
    ConfigReader r;
    out->width = r.size(cfg, "", "width"), out->vocab = r.size(cfg, "", "vocab"), out->max_positions = r.size(cfg, "", "max_positions");
    out->eps = r.number(*r.object(cfg, "", "norm"), "norm.", "eps");
    out->embed_scale = r.number(*r.object(cfg, "", "embedding"), "embedding.", "scale");
    out->embed = "embed", out->head = "embed", out->pos = "pos", out->out_norm = "final.norm";
    const JsonValue* layers = cfg.get("layers");
    if (layers == nullptr || !layers->is(JsonValue::kArray) || layers->items.empty()) return "config.json: layers is missing or empty";
    for (size_t i = 0; i < layers->items.size(); ++i) {
        const JsonValue& e = layers->items[i];
        const std::string where = "layers[" + std::to_string(i) + "].", p = "l" + std::to_string(i) + ".", m = p + "mix.";
        const std::string type = r.text(e, where, "type");
        const JsonValue& mx = *r.object(e, where, "mixer");
        LayerSpec ly;
        ly.parallel = true;
        MixerSpec l;
        l.heads = r.size(mx, where + "mixer.", "heads"), l.vdim = r.size(mx, where + "mixer.", "vdim");
        if (type == "mamba2") {
            l.kind = MixerKind::kMamba2;
            l.state = r.size(mx, where + "mixer.", "state"), l.groups = r.size(mx, where + "mixer.", "groups");
            l.conv = r.size(mx, where + "mixer.", "conv"), l.norm_groups = r.size(mx, where + "mixer.", "norm_groups");
            l.in = {m + "in"};
            l.conv_w = m + "conv", l.conv_b = m + "conv.b", l.dt_bias = m + "dt_bias", l.a_log = m + "A_log", l.d_skip = m + "D", l.mix_norm = m + "norm";
        } else if (type == "hgrn2") {
            l.kind = MixerKind::kHgrn2;
            l.dim = r.size(mx, where + "mixer.", "dim");
            l.in = {m + "q", m + "f", m + "v"};
            l.f_bias = m + "f.b", l.lower = m + "lower", l.mix_norm = m + "norm";
        } else if (type == "attention") {
            l.kind = MixerKind::kAttention;
            l.dim = r.size(mx, where + "mixer.", "dim"), l.kv_heads = r.size(mx, where + "mixer.", "kv_heads"), l.scale = r.number(mx, where + "mixer.", "scale");
            const JsonValue& mask = *r.object(mx, where + "mixer.", "mask");
            l.window = r.size(mask, where + "mixer.mask.", "size"), l.pool = r.size(mask, where + "mixer.mask.", "pool");
            l.head_gate = true;
            l.in = {m + "q", m + "k", m + "v", m + "g"};
        } else {
            return "config.json: " + where + "type '" + type + "' is unknown";
        }
        l.out = m + "o", ly.norm1 = p + "norm1";
        ly.mixers.push_back(std::move(l));
        ly.gated_residual = true, ly.gate1 = p + "rg1", ly.gate1_bias = p + "rg1.b";
        const JsonValue* mlp = e.get("mlp");
        if (mlp != nullptr && !mlp->is(JsonValue::kNull)) {
            if (!mlp->is(JsonValue::kObject)) return "config.json: " + where + "mlp is not an object";
            const std::string kind = r.text(*mlp, where + "mlp.", "kind");
            if (kind != "dense") return "config.json: " + where + "mlp.kind '" + kind + "' is unknown";
            ly.ff_kind = FfKind::kDense, ly.ff = r.size(*mlp, where + "mlp.", "ff");
            ly.norm2 = p + "norm2", ly.gate2 = p + "rg2", ly.gate2_bias = p + "rg2.b";
            ly.ff_gate = p + "mlp.gate", ly.ff_up = p + "mlp.up", ly.ff_down = p + "mlp.down";
        }
        out->layers.push_back(std::move(ly));
    }
    return r.error;
}

// The retention mixer of Tosevik; m: prefix of its tensors.
inline MixerSpec read_retention(ConfigReader& r, const JsonValue& v, const std::string& where, const std::string& m) {
    MixerSpec x;
    x.kind = MixerKind::kRetention;
    x.heads = r.size(v, where, "heads"), x.dim = r.size(v, where, "dim"), x.vdim = r.size(v, where, "vdim");
    if (const JsonValue* rot = r.optional(v, where, "rot")) x.rot_dims = r.size(*rot, where + "rot.", "dims"), x.rot_base = r.real(*rot, where + "rot.", "base");
    const JsonValue* decay = v.get("decay");
    if (decay == nullptr || !decay->is(JsonValue::kArray) || decay->items.size() != static_cast<size_t>(x.heads)) {
        r.fail_key(where, "decay", "is not a list of one number per head");
    } else {
        for (const JsonValue& d : decay->items) {
            if (!d.is(JsonValue::kNumber) || !(d.number() >= 0.0 && d.number() <= 1.0)) r.fail_key(where, "decay", "holds something other than numbers from 0 to 1");
            else x.decay.push_back(static_cast<float>(d.number()));
        }
    }
    x.in = {m + "q", m + "k", m + "v", m + "g"}, x.out = m + "o";
    return x;
}
// The attention of Tosevik: weights sigmoid(score - slope * distance + bias) over every earlier key, norms of queries, keys and values.
inline MixerSpec read_logistic(ConfigReader& r, const JsonValue& v, const std::string& where, const std::string& m) {
    MixerSpec x;
    x.kind = MixerKind::kLogistic;
    x.heads = r.size(v, where, "heads"), x.kv_heads = r.size(v, where, "kv_heads"), x.dim = r.size(v, where, "dim"), x.vdim = r.size(v, where, "vdim");
    x.scale = r.number(v, where, "scale");
    if (const JsonValue* temp = r.optional(v, where, "q_temp")) x.temp_coef = r.number(*temp, where + "q_temp.", "coef"), x.temp_every = r.number(*temp, where + "q_temp.", "every");
    if (!(x.temp_every > 0.0f)) r.fail_key(where + "q_temp.", "every", "is not positive");
    x.value_norm = true, x.distance_bias = true;
    x.in = {m + "q", m + "k", m + "v"}, x.out = m + "o";
    x.q_norm = m + "q.norm", x.k_norm = m + "k.norm", x.logit_bias = m + "pb";
    return x;
}

// Tosevik: mixer, then mixture of experts; mixers retention, and attention with logistic weights beside retention; norms tanh(alpha x) w + b;
// what a layer passes on is a weighted sum of the embedding output and all results so far; no bound on positions; untied output table.
inline std::string read_tosevik(const JsonValue& cfg, LayeredSpec* out) {
    ConfigReader r;
    out->width = r.size(cfg, "", "width"), out->vocab = r.size(cfg, "", "vocab");
    out->eps = r.number(*r.object(cfg, "", "norm"), "norm.", "eps");
    out->norm = NormKind::kTanh;
    out->embed = "embed", out->embed_norm = "embed.norm", out->head = "head", out->out_norm = "final.norm";
    const JsonValue* layers = cfg.get("layers");
    if (layers == nullptr || !layers->is(JsonValue::kArray) || layers->items.empty()) return "config.json: layers is missing or empty";
    for (size_t i = 0; i < layers->items.size(); ++i) {
        const JsonValue& e = layers->items[i];
        const std::string where = "layers[" + std::to_string(i) + "].", p = "l" + std::to_string(i) + ".", m = p + "mix.";
        const std::string type = r.text(e, where, "type");
        const JsonValue& mx = *r.object(e, where, "mixer");
        LayerSpec l;
        if (type == "retention") {
            l.mixers.push_back(read_retention(r, mx, where + "mixer.", m));
        } else if (type == "parallel") {
            l.mixers.push_back(read_logistic(r, *r.object(mx, where + "mixer.", "left"), where + "mixer.left.", m + "left."));
            l.mixers.push_back(read_retention(r, *r.object(mx, where + "mixer.", "right"), where + "mixer.right.", m + "right."));
            l.mixers[0].result_norm = m + "left.out", l.mixers[1].result_norm = m + "right.out";
        } else {
            return "config.json: " + where + "type '" + type + "' is unknown";
        }
        l.norm1 = p + "norm1", l.depth = p + "dwa";
        const JsonValue* mlp = e.get("mlp");
        if (mlp != nullptr && !mlp->is(JsonValue::kNull)) {
            if (!mlp->is(JsonValue::kObject)) return "config.json: " + where + "mlp is not an object";
            const std::string kind = r.text(*mlp, where + "mlp.", "kind"), f = p + "mlp.";
            if (kind != "moe") return "config.json: " + where + "mlp.kind '" + kind + "' is unknown";
            const JsonValue& router = *r.object(*mlp, where + "mlp.", "router");
            l.ff_kind = FfKind::kExperts, l.norm2 = p + "norm2";
            l.ff = r.size(*r.object(*mlp, where + "mlp.", "expert"), where + "mlp.expert.", "ff");
            l.shared_ff = r.size(*r.object(*mlp, where + "mlp.", "shared"), where + "mlp.shared.", "ff");
            l.experts = r.size(router, where + "mlp.router.", "experts"), l.top = r.size(router, where + "mlp.router.", "top");
            l.router_scale = r.number(router, where + "mlp.router.", "scale");
            if (const JsonValue* g = r.optional(router, where + "mlp.router.", "groups"))
                l.expert_groups = r.size(*g, where + "mlp.router.groups.", "count"), l.keep_groups = r.size(*g, where + "mlp.router.groups.", "keep");
            l.expert_prefix = f + "e", l.router = f + "router";
            l.shared_gate = f + "shared.gate", l.shared_up = f + "shared.up", l.shared_down = f + "shared.down", l.shared_scale = f + "shared.sg";
        }
        out->layers.push_back(std::move(l));
    }
    return r.error;
}

struct LayeredDesign {
    const char* architecture;  // config.json "architecture"
    std::string (*read)(const JsonValue& config, LayeredSpec* out);  // returns what is wrong, or an empty string
};
inline const LayeredDesign kLayeredDesigns[] = {{"Lasosun", read_lasosun}, {"Tosevik", read_tosevik}};

// What the kernels ask of the sizes; returns what is wrong, or an empty string.
inline std::string check_layered(const LayeredSpec& s) {
    for (size_t i = 0; i < s.layers.size(); ++i) {
        const LayerSpec& ly = s.layers[i];
        const std::string at = "layer " + std::to_string(i) + ": ";
        for (const MixerSpec& l : ly.mixers) {
            if (l.kind == MixerKind::kMamba2) {
                if (l.heads % l.groups != 0) return at + "heads is not a multiple of groups";
                if (l.inner() % l.norm_groups != 0) return at + "norm_groups does not divide heads * vdim";
            }
            if (!l.cached() && l.key_dim() > 256) return at + "more than 256 state rows per head";
            if (l.cached()) {
                if (l.heads % l.kv_heads != 0) return at + "heads is not a multiple of kv_heads";
                if (l.dim > 256 || l.vdim > 256) return at + "attention heads of more than 256 dimensions";
            }
            if (l.rot_dims % 2 != 0 || l.rot_dims > l.dim) return at + "rot.dims is odd or larger than dim";
        }
        if (ly.ff_kind == FfKind::kExperts) {
            if (ly.experts > 1024) return at + "more than 1024 experts";
            if (ly.experts % ly.expert_groups != 0) return at + "groups.count does not divide the number of experts";
            if (ly.keep_groups > ly.expert_groups) return at + "groups.keep is larger than groups.count";
            if (ly.top > ly.experts / ly.expert_groups * ly.keep_groups) return at + "top is larger than the number of experts that can be chosen";
            if (ly.top > 32) return at + "more than 32 experts per token";
        }
    }
    return "";
}

// A folder with config.json and model.safetensors; QUINTRIT_OK or an error of the C ABI.
inline int read_model_folder(const std::string& dir, LayeredSpec* spec, SafetensorsFile* file) {
    std::ifstream in(dir + "/config.json", std::ios::binary);
    if (!in) return fail(QUINTRIT_ERR_IO, "cannot open %s/config.json", dir.c_str());
    std::stringstream buf;
    buf << in.rdbuf();
    const std::string text = buf.str();
    JsonValue cfg;
    std::string why;
    if (!JsonReader(text.data(), text.size()).parse(&cfg, &why) || !cfg.is(JsonValue::kObject)) return fail(QUINTRIT_ERR_FORMAT, "config.json is not a JSON object (%s)", why.c_str());
    const JsonValue* arch = cfg.get("architecture");
    if (arch == nullptr || !arch->is(JsonValue::kString)) return fail(QUINTRIT_ERR_MODEL, "config.json names no architecture");
    const LayeredDesign* design = nullptr;
    for (const LayeredDesign& d : kLayeredDesigns)
        if (arch->s == d.architecture) design = &d;
    if (design == nullptr) return fail(QUINTRIT_ERR_UNSUPPORTED, "the architecture '%s' is not known", arch->s.c_str());
    spec->design = design->architecture;
    if (!(why = design->read(cfg, spec)).empty()) return fail(QUINTRIT_ERR_MODEL, "%s", why.c_str());
    if (!(why = check_layered(*spec)).empty()) return fail(QUINTRIT_ERR_UNSUPPORTED, "%s", why.c_str());
    const int rc = file->open(dir + "/model.safetensors", why);
    if (rc == 1) return fail(QUINTRIT_ERR_IO, "%s", why.c_str());
    if (rc != 0) return fail(QUINTRIT_ERR_FORMAT, "%s", why.c_str());
    return QUINTRIT_OK;
}

struct LayeredFolder {
    LayeredSpec spec;
    SafetensorsFile file;
};

// The folder's directory as text: hyperparameters one per line, layers, tensors by name.
inline std::string describe_layered(const LayeredSpec& s, const SafetensorsFile& f) {
    char num[96];
    std::string t = "architecture " + s.design + "\nvocab_size " + std::to_string(s.vocab) + "\nhidden_size " + std::to_string(s.width) + "\nnum_layers " + std::to_string(s.layers.size()) +
                    "\ncontext_length " + std::to_string(s.max_positions) + "\ntied " + (s.head == s.embed ? "1" : "0") + "\n";
    std::snprintf(num, sizeof num, "rms_norm_eps %.9g\nembed_scale %.9g\n", static_cast<double>(s.eps), static_cast<double>(s.embed_scale));
    t += num;
    for (size_t i = 0; i < s.layers.size(); ++i) {
        const LayerSpec& ly = s.layers[i];
        t += "layer_" + std::to_string(i);
        for (size_t k = 0; k < ly.mixers.size(); ++k) {
            const MixerSpec& l = ly.mixers[k];
            t += std::string(k > 0 ? " | " : " ") + mixer_name(l.kind) + " heads=" + std::to_string(l.heads) + " vdim=" + std::to_string(l.vdim);
            if (l.kind == MixerKind::kMamba2)
                t += " state=" + std::to_string(l.state) + " groups=" + std::to_string(l.groups) + " conv=" + std::to_string(l.conv) + " norm_groups=" + std::to_string(l.norm_groups);
            else
                t += " dim=" + std::to_string(l.dim);
            if (l.kind == MixerKind::kAttention) {
                std::snprintf(num, sizeof num, " kv_heads=%d window=%d pool=%d scale=%.9g", l.kv_heads, l.window, l.pool, static_cast<double>(l.scale));
                t += num;
            } else if (l.kind == MixerKind::kLogistic) {
                std::snprintf(num, sizeof num, " kv_heads=%d scale=%.9g q_temp=%.9g/%.9g", l.kv_heads, static_cast<double>(l.scale), static_cast<double>(l.temp_coef), static_cast<double>(l.temp_every));
                t += num;
            } else if (l.kind == MixerKind::kRetention) {
                std::snprintf(num, sizeof num, " rot=%d/%.9g decay=", l.rot_dims, l.rot_base);
                t += num;
                for (size_t h = 0; h < l.decay.size(); ++h) {
                    std::snprintf(num, sizeof num, "%s%.9g", h > 0 ? "," : "", static_cast<double>(l.decay[h]));
                    t += num;
                }
            }
        }
        t += " ff=" + std::to_string(ly.ff);
        if (ly.ff_kind == FfKind::kExperts) {
            std::snprintf(num, sizeof num, " experts=%d top=%d groups=%d/%d router_scale=%.9g shared_ff=%d", ly.experts, ly.top, ly.keep_groups, ly.expert_groups, static_cast<double>(ly.router_scale), ly.shared_ff);
            t += num;
        }
        t += "\n";
    }
    for (const auto& e : f.tensors) {
        t += "tensor " + e.first + " type=" + e.second.dtype + " shape=";
        for (size_t i = 0; i < e.second.shape.size(); ++i) t += (i ? "x" : "") + std::to_string(e.second.shape[i]);
        t += " bytes=" + std::to_string(e.second.bytes) + "\n";
    }
    return t;
}

}  // namespace qtb
