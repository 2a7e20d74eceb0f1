// Description of a decoder whose layers differ from one another, and the registry that turns a model folder (config.json +
// model.safetensors) into one. A layer is a token mixer - a recurrence or an attention - and a feed-forward, each with its own sizes
// and constants; a design is an entry of kLayeredDesigns: it names its config keys and tensors and fills the description.
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

enum class MixerKind { kMamba2, kHgrn2, kAttention };

inline const char* mixer_name(MixerKind k) { return k == MixerKind::kMamba2 ? "mamba2" : k == MixerKind::kHgrn2 ? "hgrn2" : "attention"; }

struct LayerSpec {
    MixerKind kind = MixerKind::kAttention;
    int heads = 0;
    int dim = 0, vdim = 0;                // query / key size (hgrn2, attention) and value size of a head
    int state = 0, groups = 0;            // mamba2: state size, groups that share B and C
    int conv = 0, norm_groups = 0;        // mamba2: taps of the short convolution, parts of the output norm
    int kv_heads = 0;                     // attention
    float scale = 1.0f;                   // attention: factor of q . k
    int window = 0;                       // attention: position i sees j with 0 <= i - j < window
    int pool = 0;                         // attention: block size of the pooled keys and values before the window, 0 = none
    bool head_gate = false;               // attention: one sigmoid per head on the output
    int ff = 0;                           // feed-forward width (SwiGLU), 0 = no feed-forward
    bool gated_residual = false;          // each sublayer's result is multiplied by sigmoid(W h + b) before it is added
    // tensor names
    std::vector<std::string> in;          // projections of the mixer, stacked row-wise in the order the mixer kernels read them
    std::string out, norm1, norm2, gate1, gate1_bias, gate2, gate2_bias, ff_gate, ff_up, ff_down;
    std::string conv_w, conv_b, dt_bias, a_log, d_skip, mix_norm, f_bias, lower;

    int inner() const { return heads * vdim; }                          // width of the mixer's output before the output projection
    int conv_dim() const { return inner() + 2 * groups * state; }       // mamba2: channels of the convolution (x | B | C)
    int key_dim() const { return kind == MixerKind::kMamba2 ? state : dim; }  // rows of a head's recurrent state
    int in_rows() const {
        switch (kind) {
            case MixerKind::kMamba2: return 2 * inner() + 2 * groups * state + heads;                             // z | x | B | C | dt
            case MixerKind::kHgrn2: return 2 * heads * dim + inner();                                             // q | f | v
            default: return heads * dim + kv_heads * (dim + vdim) + (head_gate ? heads : 0);                      // q | k | v | g
        }
    }
};

struct LayeredSpec {
    std::string design;
    int width = 0, vocab = 0, max_positions = 0;
    float eps = 0.0f, embed_scale = 1.0f;
    std::vector<LayerSpec> layers;
    std::string embed, pos, head, out_norm;  // pos empty: no position vectors; head: the output table (the embedding when tied)
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
        LayerSpec l;
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
        l.out = m + "o", l.norm1 = p + "norm1";
        l.gated_residual = true, l.gate1 = p + "rg1", l.gate1_bias = p + "rg1.b";
        const JsonValue* mlp = e.get("mlp");
        if (mlp != nullptr && !mlp->is(JsonValue::kNull)) {
            if (!mlp->is(JsonValue::kObject)) return "config.json: " + where + "mlp is not an object";
            const std::string kind = r.text(*mlp, where + "mlp.", "kind");
            if (kind != "dense") return "config.json: " + where + "mlp.kind '" + kind + "' is unknown";
            l.ff = r.size(*mlp, where + "mlp.", "ff");
            l.norm2 = p + "norm2", l.gate2 = p + "rg2", l.gate2_bias = p + "rg2.b";
            l.ff_gate = p + "mlp.gate", l.ff_up = p + "mlp.up", l.ff_down = p + "mlp.down";
        }
        out->layers.push_back(std::move(l));
    }
    return r.error;
}

struct LayeredDesign {
    const char* architecture;  // config.json "architecture"
    std::string (*read)(const JsonValue& config, LayeredSpec* out);  // returns what is wrong, or an empty string
};
inline const LayeredDesign kLayeredDesigns[] = {{"Lasosun", read_lasosun}};

// What the kernels ask of the sizes; returns what is wrong, or an empty string.
inline std::string check_layered(const LayeredSpec& s) {
    for (size_t i = 0; i < s.layers.size(); ++i) {
        const LayerSpec& l = s.layers[i];
        const std::string at = "layer " + std::to_string(i) + ": ";
        if (l.kind == MixerKind::kMamba2) {
            if (l.heads % l.groups != 0) return at + "heads is not a multiple of groups";
            if (l.inner() % l.norm_groups != 0) return at + "norm_groups does not divide heads * vdim";
        }
        if (l.kind != MixerKind::kAttention && l.key_dim() > 256) return at + "more than 256 state rows per head";
        if (l.kind == MixerKind::kAttention) {
            if (l.heads % l.kv_heads != 0) return at + "heads is not a multiple of kv_heads";
            if (l.dim > 256 || l.vdim > 256) return at + "attention heads of more than 256 dimensions";
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
        const LayerSpec& l = s.layers[i];
        t += "layer_" + std::to_string(i) + " " + mixer_name(l.kind) + " heads=" + std::to_string(l.heads) + " vdim=" + std::to_string(l.vdim);
        if (l.kind == MixerKind::kMamba2)
            t += " state=" + std::to_string(l.state) + " groups=" + std::to_string(l.groups) + " conv=" + std::to_string(l.conv) + " norm_groups=" + std::to_string(l.norm_groups);
        else
            t += " dim=" + std::to_string(l.dim);
        if (l.kind == MixerKind::kAttention) {
            std::snprintf(num, sizeof num, " kv_heads=%d window=%d pool=%d scale=%.9g", l.kv_heads, l.window, l.pool, static_cast<double>(l.scale));
            t += num;
        }
        t += " ff=" + std::to_string(l.ff) + "\n";
    }
    for (const auto& e : f.tensors) {
        t += "tensor " + e.first + " type=" + e.second.dtype + " shape=";
        for (size_t i = 0; i < e.second.shape.size(); ++i) t += (i ? "x" : "") + std::to_string(e.second.shape[i]);
        t += " bytes=" + std::to_string(e.second.bytes) + "\n";
    }
    return t;
}

}  // namespace qtb
