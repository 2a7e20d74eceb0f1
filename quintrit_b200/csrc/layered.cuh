// Decoder of a layered model (layered_spec.hpp) on the device: weights, sequence store, and the launch sequences of a decode step, a
// prompt chunk and a step of several sequences. It stands behind the same decoder handle as the ternary models: token, position, history
// and logits are the decoder's own (decoder.cuh), and so are its CUDA graph, greedy choice, sampling, sessions and batches.
//
// Parallel layers (mixer and feed-forward read the same residual stream): a decode step takes three launches a layer: norms and every projection
// of their results (norm_project_kernel), the mixer, and output norm + output and down projection + gates + residual sum
// (finish_project_kernel). Many tokens take the tensor cores: norms, one product of both stacks, the mixer, its output norm, and one product of
// two accumulators that ends in the residual sum.
//
// Other layers (the feed-forward reads what the mixer left): projections, mixer or two of them, output projection (out_project_kernel), router and
// shared expert with the second norm before them, chosen experts' activations, their results with all that follows them up to the next layer
// (dense_moe.cuh). Many tokens: the same steps as products on the tensor cores with rows_kernel between them.
//
// Weights are stored in the serving type (bf16, or float when the model was opened in 32-bit mode). Rows of a stack start at multiples of
// 128 and columns are padded to 64, so that one layout serves the streaming kernels and the tensor cores.
#pragma once
#include <memory>

#include "chunk_scan.cuh"
#include "dense_gemm_tc.cuh"
#include "dense_gemv.cuh"
#include "dense_moe.cuh"
#include "gated_scan.cuh"
#include "layered_spec.hpp"
#include "logistic_attention.cuh"
#include "logistic_attention_tc.cuh"
#include "pooled_attention.cuh"
#include "pooled_attention_mma.cuh"
#include "retention_chunks.cuh"
#include "tensor_map.cuh"

namespace qtb {

constexpr int kLayeredChunk = 2048;     // tokens of a prompt chunk
constexpr int kLayeredLogitRows = 64;   // rows of logits computed at a time when several positions of a chunk are asked for
constexpr int kLayeredMaxBatch = 256;   // sequences of a batched step
constexpr uint32_t kLayeredContext = 8192;  // tokens a sequence may hold where neither the model nor the caller says

inline int round_up(int v, int m) { return (v + m - 1) / m * m; }

struct LayeredMatrix {
    void* w = nullptr;
    int rows_pad = 0, pitch = 0, cols = 0;
    CUtensorMap map{};
};
struct LayeredMixer {
    MixerSpec spec;
    int col = 0;                        // first column of its projections in a token's row
    LayeredMatrix o;
    float *conv_w = nullptr, *conv_b = nullptr, *dt_bias = nullptr, *a_log = nullptr, *d_skip = nullptr, *mix_norm = nullptr, *f_bias = nullptr, *lower = nullptr;
    float *decay = nullptr, *q_norm = nullptr, *k_norm = nullptr, *slope = nullptr, *logit_bias = nullptr, *result_norm = nullptr;
    double* turns = nullptr;
};
struct LayeredLayer {
    LayerSpec spec;
    int mixer0 = 0;                     // number of its first mixer, counted over the model
    std::vector<LayeredMixer> mix;
    LayeredMatrix in1, in2, down;       // mixer projections + gate 1; gate | up interleaved + gate 2, or router, shared scale and shared gate | up; (shared) down
    LayeredMatrix experts_in, experts_down;  // every expert's gate | up interleaved, and down, at multiples of its padded rows
    std::vector<int> row1, row2;        // first rows of the parts of the two stacks
    NormParams norm1{}, norm2{};
    float *gate1_bias = nullptr, *gate2_bias = nullptr, *depth = nullptr;
    int expert_rows() const { return experts_in.rows_pad / spec.experts; }
    int expert_down_rows() const { return experts_down.rows_pad / spec.experts; }
};
// The weights on the device, shared by every decoder of the model.
struct LayeredModel {
    LayeredSpec spec;
    bool f32 = false;
    int device = 0, sm_count = 0;
    std::vector<LayeredLayer> layers;
    LayeredMatrix embed, head;
    void* pos_table = nullptr;
    NormParams embed_norm{}, out_norm{};
    int mixers = 0, depth_vectors = 0;  // depth_vectors: the embedding output and every layer's result, where layers average over them
    std::vector<void*> allocs;
    LayeredModel() = default;
    LayeredModel(const LayeredModel&) = delete;
    LayeredModel& operator=(const LayeredModel&) = delete;
    ~LayeredModel() {
        int prev = -1;
        cudaGetDevice(&prev);
        cudaSetDevice(device);
        for (void* p : allocs) cudaFree(p);
        if (prev >= 0) cudaSetDevice(prev);
    }
    size_t elem() const { return f32 ? 4 : 2; }
    // A model whose layers keep a recurrent state cannot go back to an earlier position of a sequence, only to its start.
    bool recurrent() const {
        for (const LayeredLayer& l : layers)
            for (const LayeredMixer& x : l.mix)
                if (!x.spec.cached()) return true;
        return false;
    }
};

// What `slots` sequences hold: recurrent states (one allocation, so that a step can be timed and undone) and windowed caches.
struct LayeredStore {
    int slots = 0;
    float* recurrent = nullptr;
    size_t recurrent_floats = 0;
    struct Mixer {
        float *state = nullptr, *conv = nullptr;
        size_t state_stride = 0, conv_stride = 0;  // floats per slot
        PooledCache cache{};
        CUtensorMap kmap{}, vmap{};                // logistic attention: the cached keys and values, [slot][position][kv heads x padded dim]
    };
    std::vector<Mixer> mixers;
};

struct LayeredDecoder {
    std::shared_ptr<LayeredModel> model;
    LayeredStore store;
    float* recurrent_backup = nullptr;
    uint32_t *tokens = nullptr, *pos = nullptr, *rows = nullptr;
    float *x = nullptr, *p1 = nullptr, *g1 = nullptr, *g2 = nullptr, *y[2] = {nullptr, nullptr}, *many_logits = nullptr;  // g1, g2: gates, or the results of two mixers
    void *h1 = nullptr, *h2 = nullptr, *y_t[2] = {nullptr, nullptr}, *m = nullptr, *h_head = nullptr;
    CUtensorMap map_h1{}, map_h2{}, map_head{};
    std::vector<CUtensorMap> map_y, map_q, map_m;  // per mixer, per mixer, per layer: the pitches differ
    float *x_mid = nullptr, *past = nullptr;  // residual stream between mixer and feed-forward; vectors of the depth averages, [vector][token][width]
    void* q = nullptr;                      // normed queries
    struct Experts {                        // mixture of experts: router, chosen pairs and their activations and results
        float *logits = nullptr, *shared_scale = nullptr, *weight = nullptr;
        int *chosen = nullptr, *count = nullptr, *rank = nullptr, *first = nullptr, *n_runs = nullptr;
        uint32_t* row = nullptr;
        DenseRun *up_runs = nullptr, *down_runs = nullptr;
        void *h = nullptr, *m = nullptr, *out = nullptr;
        CUtensorMap map_h{};
        std::vector<CUtensorMap> map_m;     // per layer
    } ex;
    float *part_acc = nullptr, *part_ml = nullptr;
    unsigned int* done = nullptr;
    char* work = nullptr;               // chunked recurrences: operands of one layer (ChunkWork, RetentionWork)
};

// Where the tokens of a pass sit: consecutive tokens of one sequence (`slot` of the store, position in pos[0]), or one token for each of
// `seq`'s sequences.
struct LayeredTarget {
    const LayeredStore* store = nullptr;
    int slot = 0;
    const uint32_t* pos = nullptr;
    SeqIndex seq{nullptr, 0, 0};
    bool step() const { return seq.pos_stride != 0; }
};

// ---- loading ---------------------------------------------------------------------------------------------------------------------------
class LayeredLoader {
  public:
    LayeredLoader(LayeredModel* m, const SafetensorsFile& f) : m_(m), f_(f) {}
    int run() {
        const LayeredSpec& s = m_->spec;
        for (const LayerSpec& l : s.layers) {
            m_->layers.emplace_back();
            LayeredLayer& d = m_->layers.back();
            d.spec = l, d.mixer0 = m_->mixers;
            m_->mixers += static_cast<int>(l.mixers.size());
            if (!l.depth.empty()) m_->depth_vectors = static_cast<int>(s.layers.size()) + 1;
            if (int rc = layer(l, m_->layers.size() - 1, &d)) return rc;
        }
        if (int rc = matrix({Part{{s.embed}, s.vocab}}, s.width, &m_->embed, nullptr)) return rc;
        if (s.head == s.embed) m_->head = m_->embed;
        else if (int rc = matrix({Part{{s.head}, s.vocab}}, s.width, &m_->head, nullptr)) return rc;
        if (!s.pos.empty())
            if (int rc = table(s.pos, {uint64_t(s.max_positions), uint64_t(s.width)}, &m_->pos_table)) return rc;
        if (!s.embed_norm.empty())
            if (int rc = norm(s.embed_norm, &m_->embed_norm)) return rc;
        if (int rc = norm(s.out_norm, &m_->out_norm)) return rc;
        QTB_CUDA(cudaDeviceSynchronize());
        return QUINTRIT_OK;
    }

  private:
    LayeredModel* m_;
    const SafetensorsFile& f_;
    std::vector<uint8_t> stage_;
    // A row range of a stack: tensors one after the other, or two of them row by row in turn.
    struct Part {
        std::vector<std::string> names;
        int rows;
        bool interleave = false;
    };
    int tensor(const std::string& name, const std::vector<uint64_t>& shape, const SafeTensor** out) {
        const SafeTensor* t = f_.find(name);
        if (t == nullptr) return fail(QUINTRIT_ERR_MODEL, "Missing tensor '%s'", name.c_str());
        if (!SafetensorsFile::is_float(*t)) return fail(QUINTRIT_ERR_MODEL, "tensor '%s' has the type %s, not a floating-point one", name.c_str(), t->dtype.c_str());
        if (t->shape != shape) {
            std::string have, want;
            for (uint64_t d : t->shape) have += (have.empty() ? "" : " x ") + std::to_string(d);
            for (uint64_t d : shape) want += (want.empty() ? "" : " x ") + std::to_string(d);
            return fail(QUINTRIT_ERR_MODEL, "tensor '%s' is %s, the model needs %s", name.c_str(), have.c_str(), want.c_str());
        }
        *out = t;
        return QUINTRIT_OK;
    }
    int upload(const void* host, size_t bytes, void** out) {
        void* p = nullptr;
        QTB_CUDA(cudaMalloc(&p, std::max<size_t>(bytes, 16)));
        m_->allocs.push_back(p);
        QTB_CUDA(cudaMemcpy(p, host, bytes, cudaMemcpyHostToDevice));
        *out = p;
        return QUINTRIT_OK;
    }
    int floats(const std::string& name, const std::vector<uint64_t>& shape, float** out) {
        const SafeTensor* t = nullptr;
        if (int rc = tensor(name, shape, &t)) return rc;
        std::vector<float> v(t->elements);
        for (uint64_t i = 0; i < t->elements; ++i) v[i] = SafetensorsFile::at(*t, i);
        return upload(v.data(), v.size() * 4, reinterpret_cast<void**>(out));
    }
    int floats(const std::vector<float>& v, float** out) { return upload(v.data(), v.size() * 4, reinterpret_cast<void**>(out)); }
    int norm(const std::string& name, NormParams* out) {
        const uint64_t w = m_->spec.width;
        float *weight = nullptr, *shift = nullptr;
        if (int rc = floats(name, {w}, &weight)) return rc;
        if (m_->spec.norm == NormKind::kTanh) {
            const SafeTensor* alpha = nullptr;
            if (int rc = floats(name + ".b", {w}, &shift)) return rc;
            if (int rc = tensor(name + ".alpha", {}, &alpha)) return rc;
            out->alpha = SafetensorsFile::at(*alpha, 0);
        }
        out->w = weight, out->b = shift;
        return QUINTRIT_OK;
    }
    // One row of a tensor in the storage type.
    void row(const SafeTensor& t, uint64_t r, uint64_t cols, uint8_t* dst) const {
        if (!m_->f32 && t.dtype == "BF16") {
            std::memcpy(dst, t.data + r * cols * 2, cols * 2);
            return;
        }
        for (uint64_t c = 0; c < cols; ++c) {
            const float v = SafetensorsFile::at(t, r * cols + c);
            if (m_->f32) {
                std::memcpy(dst + c * 4, &v, 4);
            } else {
                const __nv_bfloat16 b = __float2bfloat16_rn(v);
                std::memcpy(dst + c * 2, &b, 2);
            }
        }
    }
    int table(const std::string& name, const std::vector<uint64_t>& shape, void** out) {
        const SafeTensor* t = nullptr;
        if (int rc = tensor(name, shape, &t)) return rc;
        stage_.assign(t->elements * m_->elem(), 0);
        for (uint64_t r = 0; r < shape[0]; ++r) row(*t, r, shape[1], stage_.data() + r * shape[1] * m_->elem());
        return upload(stage_.data(), stage_.size(), out);
    }
    // Stacks the parts row-wise, each part padded to kRowPad rows; first_rows (optional) receives the first row of every part.
    int matrix(const std::vector<Part>& parts, int cols, LayeredMatrix* out, std::vector<int>* first_rows) {
        int rows = 0;
        for (const Part& p : parts) rows += round_up(p.rows, kRowPad);
        out->rows_pad = rows, out->pitch = round_up(cols, kColPad), out->cols = cols;
        const size_t pitch = size_t(out->pitch) * m_->elem();
        stage_.assign(size_t(rows) * pitch, 0);
        int r0 = 0;
        for (const Part& p : parts) {
            if (first_rows != nullptr) first_rows->push_back(r0);
            int r = r0;
            std::vector<const SafeTensor*> ts;
            uint64_t sum = 0;
            for (const std::string& name : p.names) {
                const SafeTensor* t = f_.find(name);
                if (t == nullptr) return fail(QUINTRIT_ERR_MODEL, "Missing tensor '%s'", name.c_str());
                const uint64_t have = t->shape.empty() ? 0 : t->shape[0];
                if (int rc = tensor(name, {have, uint64_t(cols)}, &t)) return rc;
                ts.push_back(t), sum += have;
            }
            if (sum != uint64_t(p.rows) || (p.interleave && ts[0]->shape[0] != ts[1]->shape[0]))
                return fail(QUINTRIT_ERR_MODEL, "tensor '%s'%s: %llu rows, the model needs %d", p.names[0].c_str(), p.names.size() > 1 ? " and those stacked with it" : "",
                            static_cast<unsigned long long>(sum), p.rows);
            if (p.interleave) {
                for (uint64_t i = 0; i < ts[0]->shape[0]; ++i)
                    for (int k = 0; k < 2; ++k) row(*ts[k], i, cols, stage_.data() + size_t(r++) * pitch);
            } else {
                for (const SafeTensor* t : ts)
                    for (uint64_t i = 0; i < t->shape[0]; ++i) row(*t, i, cols, stage_.data() + size_t(r++) * pitch);
            }
            r0 += round_up(p.rows, kRowPad);
        }
        if (int rc = upload(stage_.data(), stage_.size(), &out->w)) return rc;
        return m_->f32 ? QUINTRIT_OK : tensor_map_2d_bf16(&out->map, out->w, out->pitch, rows, kDenseK, kDenseM);
    }
    int layer(const LayerSpec& l, size_t index, LayeredLayer* d) {
        const int W = m_->spec.width;
        const uint64_t w = W;
        Part projections{{}, l.in_rows()};
        for (const MixerSpec& x : l.mixers) projections.names.insert(projections.names.end(), x.in.begin(), x.in.end());
        std::vector<Part> p1{projections};
        if (l.gated_residual) p1.push_back(Part{{l.gate1}, W});
        if (int rc = matrix(p1, W, &d->in1, &d->row1)) return rc;
        if (int rc = norm(l.norm1, &d->norm1)) return rc;
        if (l.gated_residual)
            if (int rc = floats(l.gate1_bias, {w}, &d->gate1_bias)) return rc;
        if (l.ff_kind == FfKind::kDense) {
            std::vector<Part> p2{Part{{l.ff_gate, l.ff_up}, 2 * l.ff, true}};
            if (l.gated_residual) p2.push_back(Part{{l.gate2}, W});
            if (int rc = matrix(p2, W, &d->in2, &d->row2)) return rc;
            if (int rc = matrix({Part{{l.ff_down}, W}}, l.ff, &d->down, nullptr)) return rc;
            if (int rc = norm(l.norm2, &d->norm2)) return rc;
            if (l.gated_residual)
                if (int rc = floats(l.gate2_bias, {w}, &d->gate2_bias)) return rc;
        } else if (l.ff_kind == FfKind::kExperts) {
            if (int rc = matrix({Part{{l.router}, l.experts}, Part{{l.shared_scale}, 1}, Part{{l.shared_gate, l.shared_up}, 2 * l.shared_ff, true}}, W, &d->in2, &d->row2)) return rc;
            if (int rc = matrix({Part{{l.shared_down}, W}}, l.shared_ff, &d->down, nullptr)) return rc;
            if (int rc = norm(l.norm2, &d->norm2)) return rc;
            std::vector<Part> in, out;
            for (int e = 0; e < l.experts; ++e) {
                const std::string name = l.expert_prefix + std::to_string(e);
                in.push_back(Part{{name + ".gate", name + ".up"}, 2 * l.ff, true}), out.push_back(Part{{name + ".down"}, W});
            }
            if (int rc = matrix(in, W, &d->experts_in, nullptr)) return rc;
            if (int rc = matrix(out, l.ff, &d->experts_down, nullptr)) return rc;
        }
        if (!l.depth.empty())
            if (int rc = floats(l.depth, {uint64_t(index) + 2}, &d->depth)) return rc;
        int col = 0;
        for (const MixerSpec& x : l.mixers) {
            d->mix.emplace_back();
            d->mix.back().spec = x, d->mix.back().col = col;
            col += x.in_rows();
            if (int rc = mixer(x, &d->mix.back())) return rc;
        }
        return QUINTRIT_OK;
    }
    int mixer(const MixerSpec& l, LayeredMixer* d) {
        const uint64_t heads = l.heads, inner = l.inner();
        int rc = matrix({Part{{l.out}, m_->spec.width}}, l.inner(), &d->o, nullptr);
        if (rc != QUINTRIT_OK) return rc;
        if (!l.result_norm.empty() && (rc = floats(l.result_norm, {uint64_t(m_->spec.width)}, &d->result_norm)) != QUINTRIT_OK) return rc;
        if (l.kind == MixerKind::kMamba2) {
            const uint64_t ch = l.conv_dim();
            (rc = floats(l.conv_w, {ch, uint64_t(l.conv)}, &d->conv_w)) || (rc = floats(l.conv_b, {ch}, &d->conv_b)) || (rc = floats(l.dt_bias, {heads}, &d->dt_bias)) ||
                (rc = floats(l.a_log, {heads}, &d->a_log)) || (rc = floats(l.d_skip, {heads}, &d->d_skip)) || (rc = floats(l.mix_norm, {inner}, &d->mix_norm));
        } else if (l.kind == MixerKind::kHgrn2) {
            const uint64_t hd = heads * l.dim;
            (rc = floats(l.f_bias, {hd}, &d->f_bias)) || (rc = floats(l.lower, {hd}, &d->lower)) || (rc = floats(l.mix_norm, {uint64_t(l.vdim)}, &d->mix_norm));
        } else if (l.kind == MixerKind::kRetention) {
            const std::vector<double> turns = rotation_turns(l.rot_dims, l.rot_base);
            (rc = floats(l.decay, &d->decay)) || (rc = upload(turns.data(), turns.size() * sizeof(double), reinterpret_cast<void**>(&d->turns)));
        } else if (l.kind == MixerKind::kLogistic) {
            std::vector<float> slope(l.heads, 0.0f);
            for (int h = 0; l.distance_bias && h < l.heads; ++h) slope[h] = static_cast<float>(std::exp2(-8.0 * (h + 1) / l.heads));
            (rc = floats(slope, &d->slope)) || (rc = floats(l.logit_bias, {heads}, &d->logit_bias)) || (rc = floats(l.q_norm, {heads * l.dim}, &d->q_norm)) ||
                (rc = floats(l.k_norm, {uint64_t(l.kv_heads) * l.dim}, &d->k_norm));
        }
        return rc;
    }
};

inline int load_layered_model(const LayeredFolder& folder, int device, bool f32, std::shared_ptr<LayeredModel>* out) {
    auto m = std::make_shared<LayeredModel>();
    m->spec = folder.spec;
    int rc = QUINTRIT_OK;
    m->device = device, m->f32 = f32;
    QTB_CUDA(cudaSetDevice(device));
    QTB_CUDA(cudaDeviceGetAttribute(&m->sm_count, cudaDevAttrMultiProcessorCount, device));
    if ((rc = LayeredLoader(m.get(), folder.file).run()) != QUINTRIT_OK) return rc;
    *out = std::move(m);
    return QUINTRIT_OK;
}

// ---- sequence store and buffers -------------------------------------------------------------------------------------------------------------
template <typename Alloc>
int layered_store_create(const LayeredModel& m, int slots, int ctx, Alloc alloc, LayeredStore* st) {
    st->slots = slots;
    st->mixers.resize(m.mixers);
    size_t total = 0;
    for (const LayeredLayer& ly : m.layers)
        for (size_t k = 0; k < ly.mix.size(); ++k) {
            const MixerSpec& l = ly.mix[k].spec;
            LayeredStore::Mixer& s = st->mixers[ly.mixer0 + k];
            if (l.cached()) continue;
            s.state_stride = size_t(l.heads) * l.vdim * l.key_dim();
            if (l.kind == MixerKind::kMamba2) s.conv_stride = size_t(l.conv) * l.conv_dim();
            total += (s.state_stride + s.conv_stride) * slots;
        }
    int rc = alloc(reinterpret_cast<void**>(&st->recurrent), std::max<size_t>(total, 4) * sizeof(float));
    if (rc != QUINTRIT_OK) return rc;
    st->recurrent_floats = total;
    float* p = st->recurrent;
    for (const LayeredLayer& ly : m.layers)
        for (size_t k = 0; k < ly.mix.size(); ++k) {
            const MixerSpec& l = ly.mix[k].spec;
            LayeredStore::Mixer& s = st->mixers[ly.mixer0 + k];
            if (!l.cached()) {
                s.state = p, p += s.state_stride * slots;
                s.conv = p, p += s.conv_stride * slots;
                continue;
            }
            PooledCache& c = s.cache;
            c.ring = l.kind == MixerKind::kLogistic ? ctx : std::min(ctx, std::max(l.window, l.pool) + kLayeredChunk);  // (every key is seen / a window of them)
            c.blocks = l.pool > 0 ? ctx / l.pool + 1 : 0;
            const size_t dp = round_up(l.dim, 8), vp = round_up(l.vdim, 8), rows = size_t(slots) * c.ring * l.kv_heads, pools = size_t(slots) * c.blocks * l.kv_heads;
            if ((rc = alloc(&c.k, rows * dp * m.elem())) || (rc = alloc(&c.v, rows * vp * m.elem())) || (rc = alloc(&c.pk, pools * dp * m.elem())) || (rc = alloc(&c.pv, pools * vp * m.elem())))
                return rc;
            if (l.kind == MixerKind::kLogistic && !m.f32 && logistic_tc_fits(l.dim, l.vdim) &&
                ((rc = tensor_map_3d_bf16(&s.kmap, c.k, l.kv_heads * dp, c.ring, slots, 64, kLtKeys)) || (rc = tensor_map_3d_bf16(&s.vmap, c.v, l.kv_heads * vp, c.ring, slots, 64, kLtKeys))))
                return rc;
        }
    return QUINTRIT_OK;
}

inline void layered_store_view(const LayeredModel& m, const LayeredStore& st, size_t mixer, const MixerSpec& l, int slot, LayeredStore::Mixer* out) {
    *out = st.mixers[mixer];
    if (slot == 0) return;
    if (!l.cached()) {
        out->state += out->state_stride * slot, out->conv += out->conv_stride * slot;
        return;
    }
    PooledCache& c = out->cache;
    const size_t dp = round_up(l.dim, 8) * m.elem(), vp = round_up(l.vdim, 8) * m.elem(), rows = size_t(slot) * c.ring * l.kv_heads, pools = size_t(slot) * c.blocks * l.kv_heads;
    c.k = static_cast<char*>(c.k) + rows * dp, c.v = static_cast<char*>(c.v) + rows * vp;
    c.pk = static_cast<char*>(c.pk) + pools * dp, c.pv = static_cast<char*>(c.pv) + pools * vp;
}

// Shares a decode step's attention is cut into: enough blocks for the device, none below one tile of keys.
inline int attention_splits(const MixerSpec& l, int ctx, int n, int sm_count) {
    if (l.kind == MixerKind::kLogistic) {
        const int gqa = l.heads / l.kv_heads, per = logistic_heads(gqa), groups = l.kv_heads * ((gqa + per - 1) / per) * n;
        return std::max(1, std::min({(ctx + kLaKeys - 1) / kLaKeys, (sm_count + groups - 1) / groups, 64}));
    }
    const int groups = l.kv_heads * ((l.heads / l.kv_heads + kPaHeads - 1) / kPaHeads) * n;
    const int keys = std::min(ctx, l.window) + (l.pool > 0 ? ctx / l.pool : 0);
    return std::max(1, std::min({(keys + kPaTile - 1) / kPaTile, 4 * sm_count / groups, 64}));
}
typedef void (*LogisticStep)(LogisticArgs, int, int);
template <typename T, bool OWN> LogisticStep logistic_step_for(int heads) {
    return heads == 1 ? logistic_step_kernel<T, OWN, 1> : heads == 4 ? logistic_step_kernel<T, OWN, 4> : logistic_step_kernel<T, OWN, 8>;
}
// The two kernels of retention over many tokens that are compiled for the head's sizes.
struct RetentionKernels {
    void (*state)(RetentionArgs);
    void (*out)(RetentionArgs);
    size_t state_smem, out_smem;
};
template <int N> RetentionKernels retention_kernels_n(int cols) {
    return {retention_state_kernel<N>, cols == 64 ? retention_out_kernel<N, 64> : cols == 128 ? retention_out_kernel<N, 128> : retention_out_kernel<N, 256>, retention_state_smem<N>(),
            retention_out_smem<N>()};
}
inline RetentionKernels retention_kernels(int rows, int cols) {
    return rows == 32 ? retention_kernels_n<32>(cols) : rows == 64 ? retention_kernels_n<64>(cols) : rows == 128 ? retention_kernels_n<128>(cols) : retention_kernels_n<256>(cols);
}
inline bool retention_chunked(const MixerSpec& l) { return retention_rows(l.dim) != 0 && retention_cols(l.vdim) != 0; }

inline int layered_decoder_setup(quintrit_b200_decoder* d, const std::shared_ptr<LayeredModel>& model) {
    const LayeredModel& m = *model;
    LayeredDecoder* y = d->lay = new LayeredDecoder();
    y->model = model;
    auto alloc = [&](void** p, size_t bytes) { return dev_alloc(d, reinterpret_cast<char**>(p), bytes); };
    int rc = layered_store_create(m, 1, d->ctx, alloc, &y->store);
    if (rc != QUINTRIT_OK) return rc;
    const size_t C = kLayeredChunk, W = m.spec.width, wp = m.embed.pitch, e = m.elem();
    size_t work = 0, p1 = 0, inner[2] = {0, 0}, op[2] = {0, 0}, mp = kColPad, parts = 1, groups = 1, acc = 4, queries = 0;
    size_t experts = 0, top = 0, pairs_mp = 0, expert_runs = 0;
    bool gates = false, sequential = false;
    for (const LayeredLayer& ly : m.layers) {
        p1 = std::max<size_t>(p1, ly.spec.in_rows()), mp = std::max<size_t>(mp, ly.down.pitch);
        gates |= ly.spec.gated_residual || ly.mix.size() > 1, sequential |= !ly.spec.parallel;
        if (ly.spec.ff_kind == FfKind::kExperts) {
            experts = std::max<size_t>(experts, ly.spec.experts), top = std::max<size_t>(top, ly.spec.top), pairs_mp = std::max<size_t>(pairs_mp, size_t(ly.spec.top) * ly.experts_down.pitch);
            expert_runs = std::max(expert_runs, C * ly.spec.top / kF32Tile + ly.spec.experts);
        }
        for (size_t k = 0; k < ly.mix.size(); ++k) {
            const LayeredMixer& x = ly.mix[k];
            const MixerSpec& l = x.spec;
            inner[k] = std::max<size_t>(inner[k], l.inner()), op[k] = std::max<size_t>(op[k], x.o.pitch);
            if (!l.cached()) {
                ChunkWork cw;
                RetentionWork rw;
                if (m.f32) continue;
                if (l.kind == MixerKind::kRetention && retention_chunked(l)) work = std::max(work, retention_work(nullptr, l.heads, l.dim, l.vdim, kLayeredChunk, &rw));
                else if (l.kind != MixerKind::kRetention && chunk_scan_rows(l.key_dim()) != 0)
                    work = std::max(work, chunk_work(nullptr, l.kind == MixerKind::kMamba2, l.heads, l.vdim, l.key_dim(), l.groups, kLayeredChunk, &cw));
                continue;
            }
            if (l.kind == MixerKind::kLogistic) queries = std::max(queries, size_t(l.heads) * round_up(l.dim, 64));
            const int per = l.kind == MixerKind::kLogistic ? logistic_heads(l.heads / l.kv_heads) : kPaHeads;
            groups = std::max<size_t>(groups, size_t(l.kv_heads) * ((l.heads / l.kv_heads + per - 1) / per));
            for (int n = 1; n <= kLayeredMaxBatch; ++n) {
                const size_t sp = attention_splits(l, d->ctx, n, m.sm_count);
                if (sp > 1) parts = std::max(parts, n * l.heads * sp), acc = std::max(acc, n * l.heads * sp * l.vdim);
            }
        }
    }
    LayeredDecoder::Experts& x = y->ex;
    if ((rc = dev_alloc(d, &y->tokens, C)) || (rc = dev_alloc(d, &y->pos, 4)) || (rc = dev_alloc(d, &y->rows, C)) || (rc = dev_alloc(d, &y->x, C * W)) || (rc = dev_alloc(d, &y->p1, C * p1)) ||
        (rc = dev_alloc(d, &y->g1, gates ? C * W : 0)) || (rc = dev_alloc(d, &y->g2, gates ? C * W : 0)) || (rc = dev_alloc(d, &y->y[0], C * inner[0])) || (rc = dev_alloc(d, &y->y[1], C * inner[1])) ||
        (rc = alloc(&y->h1, C * wp * e)) || (rc = alloc(&y->h2, C * wp * e)) || (rc = alloc(&y->y_t[0], C * op[0] * e)) || (rc = alloc(&y->y_t[1], C * op[1] * e)) ||
        (rc = alloc(&y->m, C * mp * e)) || (rc = alloc(&y->h_head, size_t(kDenseBox) * wp * e)) || (rc = dev_alloc(d, &y->x_mid, sequential ? C * W : 0)) ||
        (rc = dev_alloc(d, &y->past, size_t(m.depth_vectors) * C * W)) || (rc = alloc(&y->q, C * queries * e)) || (rc = dev_alloc(d, &y->part_acc, acc)) ||
        (rc = dev_alloc(d, &y->part_ml, 2 * parts)) || (rc = dev_alloc(d, &y->done, groups * kLayeredMaxBatch)) || (rc = dev_alloc(d, &y->work, work)))
        return rc;
    if (top > 0 && ((rc = dev_alloc(d, &x.logits, C * experts)) || (rc = dev_alloc(d, &x.shared_scale, C)) || (rc = dev_alloc(d, &x.weight, C * top)) || (rc = dev_alloc(d, &x.chosen, C * top)) ||
                    (rc = dev_alloc(d, &x.count, experts)) || (rc = dev_alloc(d, &x.rank, C * top)) || (rc = dev_alloc(d, &x.first, experts)) || (rc = dev_alloc(d, &x.n_runs, 1)) ||
                    (rc = dev_alloc(d, &x.row, C * top)) || (rc = dev_alloc(d, &x.up_runs, expert_runs)) || (rc = dev_alloc(d, &x.down_runs, expert_runs)) || (rc = alloc(&x.h, C * top * wp * e)) ||
                    (rc = alloc(&x.m, C * pairs_mp * e)) || (rc = alloc(&x.out, C * top * W * e))))
        return rc;
    if (!m.f32) {
        if ((rc = tensor_map_2d_bf16(&y->map_h1, y->h1, m.embed.pitch, C, kDenseK, kDenseBox)) || (rc = tensor_map_2d_bf16(&y->map_h2, y->h2, m.embed.pitch, C, kDenseK, kDenseBox)) ||
            (rc = tensor_map_2d_bf16(&y->map_head, y->h_head, m.embed.pitch, kDenseBox, kDenseK, kDenseBox)))
            return rc;
        if (top > 0 && (rc = tensor_map_2d_bf16(&x.map_h, x.h, m.embed.pitch, C * top, kDenseK, kDenseBox))) return rc;
        y->map_y.resize(m.mixers), y->map_q.resize(m.mixers), y->map_m.resize(m.layers.size()), x.map_m.resize(m.layers.size());
        for (size_t i = 0; i < m.layers.size(); ++i) {
            const LayeredLayer& ly = m.layers[i];
            for (size_t k = 0; k < ly.mix.size(); ++k) {
                const MixerSpec& l = ly.mix[k].spec;
                if ((rc = tensor_map_2d_bf16(&y->map_y[ly.mixer0 + k], y->y_t[k], ly.mix[k].o.pitch, C, kDenseK, kDenseBox))) return rc;
                if (l.kind == MixerKind::kLogistic && (rc = tensor_map_2d_bf16(&y->map_q[ly.mixer0 + k], y->q, size_t(l.heads) * round_up(l.dim, 64), C, 64, kLtRows))) return rc;
            }
            y->map_m[i] = y->map_y[ly.mixer0];
            if (ly.spec.ff_kind != FfKind::kNone && (rc = tensor_map_2d_bf16(&y->map_m[i], y->m, ly.down.pitch, C, kDenseK, kDenseBox))) return rc;
            if (ly.spec.ff_kind == FfKind::kExperts && (rc = tensor_map_2d_bf16(&x.map_m[i], x.m, ly.experts_down.pitch, C * ly.spec.top, kDenseK, kDenseBox))) return rc;
        }
    }
    // shared-memory limits are a property of the kernel: set to the most a block may have
    int optin = 0;
    QTB_CUDA(cudaDeviceGetAttribute(&optin, cudaDevAttrMaxSharedMemoryPerBlockOptin, m.device));
    auto allow = [&](const void* k) -> int {
        cudaFuncAttributes fa{};
        QTB_CUDA(cudaFuncGetAttributes(&fa, k));
        QTB_CUDA(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, optin - static_cast<int>(fa.sharedSizeBytes)));
        return QUINTRIT_OK;
    };
    std::vector<const void*> kernels = {reinterpret_cast<const void*>(norm_project_kernel<bf16, kProjectRms>), reinterpret_cast<const void*>(norm_project_kernel<float, kProjectRms>),
                             reinterpret_cast<const void*>(norm_project_kernel<bf16, kProjectTanh>), reinterpret_cast<const void*>(norm_project_kernel<float, kProjectTanh>),
                             reinterpret_cast<const void*>(norm_project_kernel<bf16, kProjectAny>), reinterpret_cast<const void*>(norm_project_kernel<float, kProjectAny>),
                             reinterpret_cast<const void*>(finish_project_kernel<bf16>), reinterpret_cast<const void*>(finish_project_kernel<float>),
                             reinterpret_cast<const void*>(finish_rows_kernel<bf16>), reinterpret_cast<const void*>(finish_rows_kernel<float>),
                             reinterpret_cast<const void*>(out_project_kernel<bf16>), reinterpret_cast<const void*>(out_project_kernel<float>),
                             reinterpret_cast<const void*>(rows_kernel<bf16>), reinterpret_cast<const void*>(rows_kernel<float>),
                             reinterpret_cast<const void*>(embed_norm_kernel<bf16>), reinterpret_cast<const void*>(embed_norm_kernel<float>),
                             reinterpret_cast<const void*>(moe_up_step_kernel<bf16>), reinterpret_cast<const void*>(moe_up_step_kernel<float>),
                             reinterpret_cast<const void*>(moe_down_step_kernel<bf16>), reinterpret_cast<const void*>(moe_down_step_kernel<float>),
                             reinterpret_cast<const void*>(gated_scan_kernel<kScanMamba2>), reinterpret_cast<const void*>(gated_scan_kernel<kScanHgrn2>),
                             reinterpret_cast<const void*>(gated_scan_kernel<kScanRetention>),
                             reinterpret_cast<const void*>(pooled_attention_kernel<bf16, true>), reinterpret_cast<const void*>(pooled_attention_kernel<bf16, false>),
                             reinterpret_cast<const void*>(pooled_attention_kernel<float, true>), reinterpret_cast<const void*>(pooled_attention_kernel<float, false>),
                             reinterpret_cast<const void*>(dense_gemm_tc_kernel<128, kDenseDual>), reinterpret_cast<const void*>(dense_gemm_tc_kernel<128, kDensePlain>),
                             reinterpret_cast<const void*>(dense_gemm_tc_kernel<256, kDensePlain>), reinterpret_cast<const void*>(dense_gemm_tc_kernel<128, kDenseGrouped>),
                             reinterpret_cast<const void*>(dense_gemm_tc_kernel<256, kDenseGrouped>),
                             reinterpret_cast<const void*>(chunk_scan_kernel<kScanMamba2, 32>), reinterpret_cast<const void*>(chunk_scan_kernel<kScanMamba2, 64>),
                             reinterpret_cast<const void*>(chunk_scan_kernel<kScanMamba2, 128>), reinterpret_cast<const void*>(chunk_scan_kernel<kScanHgrn2, 32>),
                             reinterpret_cast<const void*>(chunk_scan_kernel<kScanHgrn2, 64>), reinterpret_cast<const void*>(chunk_scan_kernel<kScanHgrn2, 128>),
                             reinterpret_cast<const void*>(pooled_attention_mma_kernel<32>), reinterpret_cast<const void*>(pooled_attention_mma_kernel<64>),
                             reinterpret_cast<const void*>(pooled_attention_mma_kernel<128>)};
    for (int heads : {1, 4, 8})
        for (LogisticStep k : {logistic_step_for<bf16, true>(heads), logistic_step_for<float, true>(heads), logistic_step_for<float, false>(heads)}) kernels.push_back(reinterpret_cast<const void*>(k));
    kernels.push_back(reinterpret_cast<const void*>(logistic_mma_kernel<kLogisticMmaDims>)), kernels.push_back(reinterpret_cast<const void*>(logistic_tc_kernel));
    for (int rows : {32, 64, 128, 256}) {
        kernels.push_back(reinterpret_cast<const void*>(retention_kernels(rows, 64).state));
        for (int cols : {64, 128, 256}) kernels.push_back(reinterpret_cast<const void*>(retention_kernels(rows, cols).out));
    }
    for (const void* k : kernels)
        if ((rc = allow(k)) != QUINTRIT_OK) return rc;
    // the largest requests of this model against what a block may have
    const size_t limit = static_cast<size_t>(optin) - 4608;  // (a kernel's own shared variables count too)
    for (const LayeredLayer& ly : m.layers) {
        size_t need = std::max<size_t>({3 * wp * 4, (size_t(ly.mix[0].o.pitch) + (ly.mix.size() > 1 ? ly.mix[1].o.pitch : ly.down.pitch)) * 4});
        if (!ly.spec.parallel) need = std::max(need, (size_t(ly.mix[0].o.pitch) + 2 * (ly.mix.size() > 1 ? ly.mix[1].o.pitch : ly.mix[0].o.pitch)) * 4);
        if (ly.spec.ff_kind == FfKind::kExperts) need = std::max({need, (size_t(ly.spec.top) * ly.experts_down.pitch + ly.down.pitch) * 4, (wp + 8 * size_t(ly.spec.experts)) * 4});
        for (const LayeredMixer& x : ly.mix) {
            const MixerSpec& l = x.spec;
            need = std::max(need, size_t(l.inner()) * 4);
            if (l.kind == MixerKind::kAttention) need = std::max(need, pooled_attn_smem(round_up(l.dim, 8), round_up(l.vdim, 8), static_cast<int>(e)));
            else if (l.kind == MixerKind::kLogistic) need = std::max(need, logistic_step_smem(logistic_heads(l.heads / l.kv_heads), round_up(l.dim, 8), l.vdim, round_up(l.vdim, 8), static_cast<int>(e)));
            else need = std::max(need, scan_smem(l.key_dim()));
        }
        if (need > limit) return fail(QUINTRIT_ERR_UNSUPPORTED, "a vector of the model does not fit the shared memory of one block (%zu bytes, %zu are available)", need, limit);
    }
    QTB_CUDA(cudaDeviceSynchronize());
    return QUINTRIT_OK;
}

void layered_release(quintrit_b200_decoder* d) {
    delete d->lay;
    d->lay = nullptr;
}

// ---- launch sequences -----------------------------------------------------------------------------------------------------------------------
inline DenseStack layered_stack(const LayeredMatrix& w) {
    DenseStack s{};
    s.w = w.w, s.pitch = w.pitch, s.cols = w.cols;
    return s;
}

template <typename T> void (*layered_project_kernel(const NormProjectArgs& a))(NormProjectArgs) {
    if (a.pair.r[0] != nullptr || (a.norm[0].b == nullptr && a.h_out != nullptr)) return norm_project_kernel<T, kProjectAny>;
    return a.norm[0].b != nullptr ? norm_project_kernel<T, kProjectTanh> : norm_project_kernel<T, kProjectRms>;
}

// The two stacks of a layer's projections with their endings; returns how many there are.
inline int layered_in_stacks(const LayeredDecoder& y, const LayeredLayer& l, DenseStack (&st)[2]) {
    const int W = y.model->spec.width, rows = l.spec.in_rows();
    st[0] = layered_stack(l.in1);
    st[0].seg[st[0].n_seg++] = DenseSeg{0, rows, kSegPlain, rows, y.p1, nullptr, nullptr};
    if (l.spec.gated_residual) st[0].seg[st[0].n_seg++] = DenseSeg{l.row1[1], W, kSegSigmoid, W, y.g1, nullptr, l.gate1_bias};
    if (l.spec.ff_kind == FfKind::kNone) return 1;
    st[1] = layered_stack(l.in2);
    if (l.spec.ff_kind == FfKind::kExperts) {
        st[1].seg[st[1].n_seg++] = DenseSeg{l.row2[0], l.spec.experts, kSegPlain, l.spec.experts, y.ex.logits, nullptr, nullptr};
        st[1].seg[st[1].n_seg++] = DenseSeg{l.row2[1], 1, kSegSigmoid, 1, y.ex.shared_scale, nullptr, nullptr};
        st[1].seg[st[1].n_seg++] = DenseSeg{l.row2[2], 2 * l.spec.shared_ff, kSegSwiGlu, l.down.pitch, nullptr, y.m, nullptr};
        return 2;
    }
    st[1].seg[st[1].n_seg++] = DenseSeg{0, 2 * l.spec.ff, kSegSwiGlu, l.down.pitch, nullptr, y.m, nullptr};
    if (l.spec.gated_residual) st[1].seg[st[1].n_seg++] = DenseSeg{l.row2[1], W, kSegSigmoid, W, y.g2, nullptr, l.gate2_bias};
    return 2;
}

inline int layered_norm_parts(const MixerSpec& l) { return l.kind == MixerKind::kMamba2 ? l.norm_groups : l.kind == MixerKind::kHgrn2 || l.kind == MixerKind::kRetention ? l.heads : 0; }
inline int layered_norm_len(const MixerSpec& l) { return l.kind == MixerKind::kMamba2 ? l.inner() : l.vdim; }

// Many tokens of retention in 64-token chunks; ends with the normed and gated output in the storage type.
inline int layered_retention_chunks(quintrit_b200_decoder* d, const MixerSpec& l, const ScanArgs& a, int k, int out_pitch) {
    RetentionArgs r{};
    r.scan = a, r.eps = d->eps, r.out = d->lay->y_t[k], r.out_pitch = out_pitch;
    retention_work(d->lay->work, l.heads, l.dim, l.vdim, a.tokens, &r.work);
    const RetentionKernels f = retention_kernels(r.work.rows, r.work.v_pad);
    const int chunks = retention_chunks(a.tokens);
    r.pairs = l.dim % 2 == 0 && l.vdim % 2 == 0 && l.rot_dims % 4 == 0 && a.ld % 2 == 0 && (a.p - d->lay->p1) % 2 == 0;
    const dim3 grid((l.heads + 3) / 4, r.work.tokens / kRetPrep);
    r.pairs ? retention_prepare_kernel<true><<<grid, 256, 0, d->stream>>>(r) : retention_prepare_kernel<false><<<grid, 256, 0, d->stream>>>(r);
    QTB_LAUNCH_CHECK();
    f.state<<<dim3(l.heads, chunks, r.work.v_pad / kRetV), 128, f.state_smem, d->stream>>>(r);
    QTB_LAUNCH_CHECK();
    retention_carry_kernel<<<dim3(r.work.v_pad * r.work.rows / 512, l.heads), 128, 0, d->stream>>>(r);
    QTB_LAUNCH_CHECK();
    f.out<<<dim3(l.heads, chunks), 128, f.out_smem, d->stream>>>(r);
    QTB_LAUNCH_CHECK();
    return QUINTRIT_OK;
}

// Many tokens of a recurrence in 16-token chunks.
inline int layered_chunk_scan(quintrit_b200_decoder* d, const MixerSpec& l, const ScanArgs& a) {
    cudaStream_t s = d->stream;
    const bool mamba = l.kind == MixerKind::kMamba2;
    ChunkWork w;
    chunk_work(d->lay->work, mamba, l.heads, l.vdim, a.n, l.groups, a.tokens, &w);
    const int chunks = chunk_count(a.tokens), rows = w.rows;
    if (mamba) {
        const dim3 cgrid((l.heads * w.v_pad + 2 * l.groups * rows + 127) / 128, chunks);
        auto conv = [&](auto kernel) { kernel<<<cgrid, 128, 0, s>>>(a, w); };
        l.conv == 4 ? conv(ssd_conv_kernel<4>) : l.conv == 3 ? conv(ssd_conv_kernel<3>) : l.conv == 2 ? conv(ssd_conv_kernel<2>) : conv(ssd_conv_kernel<0>);
        QTB_LAUNCH_CHECK();
        ssd_gram_kernel<<<dim3(l.groups + 1, chunks), 256, size_t(2 * kChunkT) * (rows + 1) * sizeof(float), s>>>(a, w);
        QTB_LAUNCH_CHECK();
    } else {
        auto prep = [&](auto kernel) { kernel<<<dim3(l.heads, chunks), 128, size_t(3 * kChunkT) * rows * sizeof(float), s>>>(a, w); };
        rows == 32 ? prep(hgrn_prep_kernel<32>) : rows == 64 ? prep(hgrn_prep_kernel<64>) : prep(hgrn_prep_kernel<128>);
        QTB_LAUNCH_CHECK();
    }
    const dim3 grid(l.heads, w.v_pad / kChunkV);
    auto go = [&](auto kernel, size_t smem) { kernel<<<grid, 128, smem, s>>>(a, w); };
    if (mamba) {
        const size_t smem = chunk_scan_smem<kScanMamba2>(rows);
        rows == 32 ? go(chunk_scan_kernel<kScanMamba2, 32>, smem) : rows == 64 ? go(chunk_scan_kernel<kScanMamba2, 64>, smem) : go(chunk_scan_kernel<kScanMamba2, 128>, smem);
        QTB_LAUNCH_CHECK();
        conv_tail_kernel<<<(l.conv_dim() + 255) / 256, 256, 0, s>>>(a);
    } else {
        const size_t smem = chunk_scan_smem<kScanHgrn2>(rows);
        rows == 32 ? go(chunk_scan_kernel<kScanHgrn2, 32>, smem) : rows == 64 ? go(chunk_scan_kernel<kScanHgrn2, 64>, smem) : go(chunk_scan_kernel<kScanHgrn2, 128>, smem);
    }
    QTB_LAUNCH_CHECK();
    return QUINTRIT_OK;
}

constexpr unsigned int kDenseSpinLimit = 1u << 16;  // polls of up to 20 us each: about a second before a wait gives up

// Mixer k of a layer over the projections in y.p1. *ready: its output is in y.y_t[k], normed, gated and in the storage type, not in y.y[k].
template <typename T>
int layered_mixer(quintrit_b200_decoder* d, size_t li, int k, int n, const LayeredTarget& tg, bool* ready) {
    LayeredDecoder& y = *d->lay;
    const LayeredLayer& ly = y.model->layers[li];
    const LayeredMixer& w = ly.mix[k];
    const MixerSpec& l = w.spec;
    cudaStream_t s = d->stream;
    LayeredStore::Mixer st;
    layered_store_view(*y.model, *tg.store, ly.mixer0 + k, l, tg.slot, &st);
    const int tokens = tg.step() ? 1 : n, seqs = tg.step() ? n : 1, ld = ly.spec.in_rows();
    const float* p = y.p1 + w.col;
    *ready = false;
    if (!l.cached()) {
        ScanArgs a{};
        a.tokens = tokens, a.pos = tg.pos, a.seq = tg.seq, a.p = p, a.ld = ld;
        a.heads = l.heads, a.vdim = l.vdim, a.n = l.key_dim(), a.groups = l.groups, a.taps = l.conv;
        a.conv_w = w.conv_w, a.conv_b = w.conv_b, a.dt_bias = w.dt_bias, a.a_log = w.a_log, a.d_skip = w.d_skip, a.f_bias = w.f_bias, a.lower = w.lower;
        a.decay = w.decay, a.turns = w.turns, a.rot_dims = l.rot_dims;
        a.state = st.state, a.conv = st.conv, a.y = y.y[k];
        const dim3 grid(l.heads, (l.vdim + kScanRows - 1) / kScanRows, seqs);
        if (l.kind == MixerKind::kRetention) {
            if (sizeof(T) == 2 && tokens > 1 && retention_chunked(l)) {
                *ready = true;
                return layered_retention_chunks(d, l, a, k, w.o.pitch);
            }
            launch_dependent(gated_scan_kernel<kScanRetention>, grid, kScanThreads, scan_smem(a.n), s, a);
            QTB_LAUNCH_CHECK();
            return QUINTRIT_OK;
        }
        if (sizeof(T) == 2 && tokens > kChunkT / 2 && chunk_scan_rows(a.n) != 0) return layered_chunk_scan(d, l, a);
        if (l.kind == MixerKind::kMamba2) {
            launch_dependent(gated_scan_kernel<kScanMamba2>, grid, kScanThreads, scan_smem(a.n), s, a);
            QTB_LAUNCH_CHECK();
            if (tokens > 1) {
                conv_tail_kernel<<<(l.conv_dim() + 255) / 256, 256, 0, s>>>(a);
                QTB_LAUNCH_CHECK();
            }
        } else {
            launch_dependent(gated_scan_kernel<kScanHgrn2>, grid, kScanThreads, scan_smem(a.n), s, a);
            QTB_LAUNCH_CHECK();
        }
        return QUINTRIT_OK;
    }
    if (l.kind == MixerKind::kLogistic) {
        LogisticArgs a{};
        a.tokens = tokens, a.pos = tg.pos, a.seq = tg.seq, a.p = p, a.ld = ld;
        a.heads = l.heads, a.kv_heads = l.kv_heads, a.dim = l.dim, a.vdim = l.vdim, a.dim_pad = round_up(l.dim, 8), a.vdim_pad = round_up(l.vdim, 8);
        a.scale = l.scale, a.eps = d->eps, a.q_norm = w.q_norm, a.k_norm = w.k_norm, a.temp_coef = l.temp_coef, a.temp_every = l.temp_every, a.value_norm = l.value_norm;
        a.slope = w.slope, a.bias = w.logit_bias, a.q = y.q, a.q_pad = round_up(l.dim, 64), a.k = st.cache.k, a.v = st.cache.v, a.capacity = st.cache.ring;
        a.out = y.y_t[k], a.out_pitch = w.o.pitch, a.y = y.y[k], a.part = y.part_acc, a.done = y.done;
        const int gqa = l.heads / l.kv_heads, per = logistic_heads(gqa), hg = l.kv_heads * ((gqa + per - 1) / per), elem = sizeof(T);
        const size_t smem = logistic_step_smem(per, a.dim_pad, a.vdim, a.vdim_pad, elem);
        const int key_lanes = std::min(logistic_lanes(a.dim_pad * elem / 16), 32), value_lanes = logistic_lanes(a.vdim_pad * elem / 16);
        if (tokens == 1) {
            a.splits = attention_splits(l, d->ctx, n, y.model->sm_count);
            launch_dependent(logistic_step_for<T, true>(per), dim3(hg, a.splits, n), kLaThreads, smem, s, a, key_lanes, value_lanes);
            QTB_LAUNCH_CHECK();
            return QUINTRIT_OK;
        }
        logistic_prepare_kernel<T><<<n + (sizeof(T) == 2 ? kLtKeys - 1 : 0), 256, 0, s>>>(a);
        QTB_LAUNCH_CHECK();
        if constexpr (sizeof(T) == 2) {
            if (logistic_tc_fits(l.dim, l.vdim)) {
                LogisticTcArgs t{};
                t.a = a, t.k_slices = logistic_tc_slices(l.dim), t.v_slices = logistic_tc_slices(l.vdim), t.slot = tg.slot, t.status = d->d_counters + 2, t.spin_limit = kDenseSpinLimit;
                logistic_tc_kernel<<<dim3((tokens + kLtRows - 1) / kLtRows, l.heads), kLtThreads, logistic_tc_smem(l.dim, l.vdim), s>>>(y.map_q[ly.mixer0 + k], st.kmap, st.vmap, t);
            } else {
                logistic_mma_kernel<kLogisticMmaDims><<<dim3((tokens + kPmRows - 1) / kPmRows, l.heads), kPmThreads, pooled_mma_smem(kLogisticMmaDims), s>>>(a);
            }
            *ready = true;
        } else {
            a.splits = 1;
            logistic_step_for<T, false>(per)<<<dim3(hg, 1, n), kLaThreads, smem, s>>>(a, key_lanes, value_lanes);
        }
        QTB_LAUNCH_CHECK();
        return QUINTRIT_OK;
    }
    PooledAttnArgs a{};
    a.tokens = tokens, a.pos = tg.pos, a.seq = tg.seq, a.p = p, a.ld = ld;
    a.heads = l.heads, a.kv_heads = l.kv_heads, a.dim = l.dim, a.vdim = l.vdim, a.dim_pad = round_up(l.dim, 8), a.vdim_pad = round_up(l.vdim, 8);
    a.window = l.window, a.pool = l.pool, a.scale = l.scale, a.head_gate = l.head_gate, a.cache = st.cache, a.y = y.y[k];
    a.part_acc = y.part_acc, a.part_ml = y.part_ml, a.done = y.done;
    const int hg = l.kv_heads * ((l.heads / l.kv_heads + kPaHeads - 1) / kPaHeads);
    const size_t smem = pooled_attn_smem(a.dim_pad, a.vdim_pad, sizeof(T));
    if (tokens == 1) {  // a token at a time: the attention kernel appends to the cache itself
        a.splits = attention_splits(l, d->ctx, n, y.model->sm_count);
        launch_dependent(pooled_attention_kernel<T, true>, dim3(hg, a.splits, seqs), kPaThreads, smem, s, a);
        QTB_LAUNCH_CHECK();
        return QUINTRIT_OK;
    }
    const int unit = l.pool > 0 ? l.pool : 64;
    pooled_append_kernel<T><<<dim3(tokens / unit + 2, l.kv_heads, 1), 256, 0, s>>>(a);
    QTB_LAUNCH_CHECK();
    a.splits = 1;
    if constexpr (sizeof(T) == 2) {
        const int dims = pooled_mma_dims(l.dim, l.vdim);
        if (dims != 0) {
            const dim3 grid((tokens + kPmRows - 1) / kPmRows, l.heads);
            auto go = [&](auto kernel) { kernel<<<grid, kPmThreads, pooled_mma_smem(dims), s>>>(a); };
            dims == 32 ? go(pooled_attention_mma_kernel<32>) : dims == 64 ? go(pooled_attention_mma_kernel<64>) : go(pooled_attention_mma_kernel<128>);
            QTB_LAUNCH_CHECK();
            return QUINTRIT_OK;
        }
    }
    pooled_attention_kernel<T, false><<<dim3(hg, 1, tokens), kPaThreads, smem, s>>>(a);
    QTB_LAUNCH_CHECK();
    return QUINTRIT_OK;
}

// Product of `n_stack` stacks over the activations h (bf16: through their tensor maps), tokens = n.
template <typename T>
int layered_gemm(quintrit_b200_decoder* d, int n, const LayeredMatrix* const (&w)[2], const CUtensorMap* const (&hmap)[2], const void* const (&h)[2], const DenseStack (&st)[2], int n_stack) {
    DenseGemmArgs a{};
    a.tokens = n, a.n_prob = n_stack, a.status = d->d_counters + 2, a.spin_limit = kDenseSpinLimit;
    int tiles = 0;
    for (int i = 0; i < n_stack; ++i) a.stack[i] = st[i], a.k_steps[i] = w[i]->pitch / kDenseK, a.row_tiles[i] = w[i]->rows_pad / kDenseM, tiles += a.row_tiles[i];
    const int j = n_stack > 1 ? 1 : 0;
    if constexpr (sizeof(T) == 2)
        if (n > kDenseBox)
            dense_gemm_tc_kernel<256, kDensePlain><<<std::min(d->sm_count, (n + 255) / 256 * tiles), kDenseThreads, dense_smem(256), d->stream>>>(w[0]->map, *hmap[0], w[j]->map, *hmap[j], a);
        else
            dense_gemm_tc_kernel<128, kDensePlain><<<std::min(d->sm_count, tiles), kDenseThreads, dense_smem(128), d->stream>>>(w[0]->map, *hmap[0], w[j]->map, *hmap[j], a);
    else
        dense_gemm_f32_kernel<kDensePlain><<<dim3((n + kF32Tile - 1) / kF32Tile, tiles * (kDenseM / kF32Tile)), 256, 0, d->stream>>>(
            static_cast<const float*>(w[0]->w), static_cast<const float*>(h[0]), w[0]->pitch, static_cast<const float*>(w[j]->w), static_cast<const float*>(h[j]), w[j]->pitch, a);
    QTB_LAUNCH_CHECK();
    return QUINTRIT_OK;
}

// x += W_o y * gate1 + W_down m * gate2 for n tokens; either product may be left out (its matrix nullptr).
template <typename T>
int layered_add(quintrit_b200_decoder* d, int n, const LayeredMatrix* o, const CUtensorMap* map_o, const void* act_o, const LayeredMatrix* down, const CUtensorMap* map_down, const void* act_down,
                DenseGemmArgs a) {
    if (o == nullptr) o = down, map_o = map_down, act_o = act_down, down = nullptr;
    a.tokens = n, a.n_prob = 1, a.status = d->d_counters + 2, a.spin_limit = kDenseSpinLimit;
    a.k_steps[0] = o->pitch / kDenseK, a.k_steps[1] = down != nullptr ? down->pitch / kDenseK : 0, a.row_tiles[0] = o->rows_pad / kDenseM;
    a.width = d->lay->model->spec.width;
    if (down == nullptr) down = o, map_down = map_o, act_down = act_o;
    if constexpr (sizeof(T) == 2)
        dense_gemm_tc_kernel<128, kDenseDual><<<std::min(d->sm_count, (n + 127) / 128 * a.row_tiles[0]), kDenseThreads, dense_smem(128), d->stream>>>(o->map, *map_o, down->map, *map_down, a);
    else
        dense_gemm_f32_kernel<kDenseDual><<<dim3((n + kF32Tile - 1) / kF32Tile, a.row_tiles[0] * (kDenseM / kF32Tile)), 256, 0, d->stream>>>(
            static_cast<const float*>(o->w), static_cast<const float*>(act_o), o->pitch, static_cast<const float*>(down->w), static_cast<const float*>(act_down), down->pitch, a);
    QTB_LAUNCH_CHECK();
    return QUINTRIT_OK;
}

// A layer whose feed-forward reads the same residual stream as its mixer, for the n tokens of y.x.
template <typename T>
int layered_parallel_layer(quintrit_b200_decoder* d, size_t li, int n, const LayeredTarget& tg) {
    LayeredDecoder& y = *d->lay;
    const LayeredModel& m = *y.model;
    const LayeredLayer& l = m.layers[li];
    const LayeredMixer& x = l.mix[0];
    cudaStream_t s = d->stream;
    const int W = m.spec.width, wp = m.embed.pitch;
    int rc;
    bool ready;
    DenseStack st[2] = {};
    const int n_stack = layered_in_stacks(y, l, st);
    const int parts = layered_norm_parts(x.spec), norm_len = layered_norm_len(x.spec);
    if (n == 1) {
        NormProjectArgs a{};
        a.x = y.x, a.norm[0] = l.norm1, a.norm[1] = l.norm2, a.eps = m.spec.eps, a.width = W, a.n_stack = n_stack;
        int units = 0;
        for (int i = 0; i < n_stack; ++i) {
            a.stack[i] = st[i];
            for (int k = 0; k < st[i].n_seg; ++k) units += (st[i].seg[k].rows + 1) / 2;
        }
        const int warps = kProjectThreads / 32;
        launch_dependent(layered_project_kernel<T>(a), dim3(std::min((units + warps - 1) / warps, 4 * m.sm_count)), kProjectThreads, size_t(n_stack) * wp * sizeof(float), s, a);
        QTB_LAUNCH_CHECK();
        if ((rc = layered_mixer<T>(d, li, 0, n, tg, &ready)) != QUINTRIT_OK) return rc;
        FinishProjectArgs f{};
        f.x = y.x, f.width = W, f.y = y.y[0], f.inner = x.spec.inner(), f.norm_parts = parts, f.norm_len = norm_len, f.norm_w = x.mix_norm, f.eps = m.spec.eps;
        f.o = x.o.w, f.o_pitch = x.o.pitch;
        if (n_stack > 1) f.m = y.m, f.down = l.down.w, f.down_pitch = l.down.pitch;
        if (l.spec.gated_residual) f.gate1 = y.g1, f.gate2 = y.g2;
        launch_dependent(finish_project_kernel<T>, dim3(std::min((W + warps - 1) / warps, 4 * m.sm_count)), kProjectThreads, (size_t(f.o_pitch) + f.down_pitch) * sizeof(float), s, f);
        QTB_LAUNCH_CHECK();
        return QUINTRIT_OK;
    }
    norm_rows_kernel<T><<<n, 256, 0, s>>>(y.x, W, m.spec.eps, l.norm1, static_cast<T*>(y.h1), l.norm2, n_stack > 1 ? static_cast<T*>(y.h2) : nullptr, wp, nullptr);
    QTB_LAUNCH_CHECK();
    const LayeredMatrix* const ws[2] = {&l.in1, &l.in2};
    const CUtensorMap* const hm[2] = {&y.map_h1, &y.map_h2};
    const void* const hs[2] = {y.h1, y.h2};
    if ((rc = layered_gemm<T>(d, n, ws, hm, hs, st, n_stack)) != QUINTRIT_OK || (rc = layered_mixer<T>(d, li, 0, n, tg, &ready)) != QUINTRIT_OK) return rc;
    const float* gate = sizeof(T) == 2 && x.spec.kind == MixerKind::kMamba2 && !tg.step() && n > kChunkT / 2 && chunk_scan_rows(x.spec.state) != 0 ? y.p1 : nullptr;  // silu(z)
    finish_rows_kernel<T><<<n, 256, size_t(x.spec.inner()) * sizeof(float), s>>>(y.y[0], gate, nullptr, l.spec.in_rows(), x.spec.inner(), parts, m.spec.eps, x.mix_norm, norm_len,
                                                                                 static_cast<T*>(y.y_t[0]), x.o.pitch);
    QTB_LAUNCH_CHECK();
    DenseGemmArgs a{};
    a.x = y.x;
    if (l.spec.gated_residual) a.gate1 = y.g1, a.gate2 = y.g2;
    return layered_add<T>(d, n, &x.o, &y.map_y[l.mixer0], y.y_t[0], n_stack > 1 ? &l.down : nullptr, &y.map_m[li], y.m, a);
}

// What a layer's result goes through on its way to the next layer.
inline DepthMix layered_depth(const LayeredDecoder& y, size_t li) {
    const LayeredModel& m = *y.model;
    if (m.layers[li].depth == nullptr) return DepthMix{nullptr, 0, nullptr, 0};
    return DepthMix{y.past, size_t(kLayeredChunk) * m.spec.width, m.layers[li].depth, static_cast<int>(li) + 2};
}

inline RouterArgs layered_router(const LayerSpec& l) { return RouterArgs{l.experts, l.expert_groups, l.keep_groups, l.top, l.router_scale}; }

// A layer whose feed-forward reads what its mixer left, one token.
template <typename T>
int layered_sequential_step(quintrit_b200_decoder* d, size_t li, const LayeredTarget& tg) {
    LayeredDecoder& y = *d->lay;
    const LayeredModel& m = *y.model;
    const LayeredLayer& l = m.layers[li];
    cudaStream_t s = d->stream;
    const int W = m.spec.width, wp = m.embed.pitch, warps = kProjectThreads / 32, sets = static_cast<int>(l.mix.size());
    int rc;
    DenseStack st[2] = {};
    layered_in_stacks(y, l, st);
    auto project = [&](NormProjectArgs a) -> int {
        int units = 0;
        for (int k = 0; k < a.stack[0].n_seg; ++k) units += (a.stack[0].seg[k].rows + 1) / 2;
        a.eps = m.spec.eps, a.width = W, a.n_stack = 1;
        launch_dependent(layered_project_kernel<T>(a), dim3(std::min((units + warps - 1) / warps, 4 * m.sm_count)), kProjectThreads, size_t(a.pair.r[0] != nullptr ? 2 : 1) * wp * sizeof(float), s, a);
        QTB_LAUNCH_CHECK();
        return QUINTRIT_OK;
    };
    NormProjectArgs a{};
    a.x = y.x, a.norm[0] = l.norm1, a.stack[0] = st[0];
    if ((rc = project(a)) != QUINTRIT_OK) return rc;
    OutProjectArgs o{};
    o.width = W, o.n = sets, o.eps = m.spec.eps;
    size_t smem = 0, gates = 0;
    for (int k = 0; k < sets; ++k) {
        const LayeredMixer& x = l.mix[k];
        bool ready;
        if ((rc = layered_mixer<T>(d, li, k, 1, tg, &ready)) != QUINTRIT_OK) return rc;
        OutProjectArgs::Mixer& t = o.mix[k];
        t.y = y.y[k], t.inner = x.spec.inner(), t.parts = layered_norm_parts(x.spec), t.w = x.o.w, t.pitch = x.o.pitch;
        if (x.spec.kind == MixerKind::kRetention) t.gate = y.p1 + x.col + x.spec.gate_col(), t.gate_ld = l.spec.in_rows();
        t.out = sets > 1 ? (k > 0 ? y.g2 : y.g1) : y.x, t.add = sets == 1;
        smem += size_t(x.o.pitch) * sizeof(float), gates = std::max(gates, t.gate != nullptr ? size_t(x.o.pitch) * sizeof(float) : 0);
    }
    smem += gates;
    launch_dependent(out_project_kernel<T>, dim3(std::min((sets * W + warps - 1) / warps, 4 * m.sm_count)), kProjectThreads, smem, s, o);
    QTB_LAUNCH_CHECK();
    PairSum pair{};
    if (sets > 1) pair = PairSum{{y.g1, y.g2}, {l.mix[0].result_norm, l.mix[1].result_norm}};
    if (l.spec.ff_kind == FfKind::kNone) {
        RowsArgs r{};
        r.x = y.x, r.x_out = y.x, r.width = W, r.pitch = wp, r.eps = m.spec.eps, r.pair = pair, r.depth = layered_depth(y, li);
        rows_kernel<T><<<1, 256, size_t(W) * sizeof(float), s>>>(r);
        QTB_LAUNCH_CHECK();
        return QUINTRIT_OK;
    }
    a = NormProjectArgs{};
    a.x = y.x, a.norm[0] = l.norm2, a.stack[0] = st[1], a.pair = pair, a.x_out = y.x_mid, a.h_out = y.h2;
    if ((rc = project(a)) != QUINTRIT_OK) return rc;
    MoeUpStepArgs u{};
    u.router = layered_router(l.spec), u.logits = y.ex.logits, u.h = y.h2, u.w = l.experts_in.w, u.pitch = l.experts_in.pitch, u.rows_pad = l.expert_rows(), u.ff = l.spec.ff;
    u.m = y.ex.m, u.m_pitch = l.experts_down.pitch, u.chosen = y.ex.chosen, u.weight = y.ex.weight;
    launch_dependent(moe_up_step_kernel<T>, dim3(std::min((l.spec.top * l.spec.ff + warps - 1) / warps, 4 * m.sm_count)), kProjectThreads, (size_t(u.pitch) + 2 * l.spec.experts) * sizeof(float), s, u);
    QTB_LAUNCH_CHECK();
    MoeDownStepArgs f{};
    f.x = sets > 1 ? y.x_mid : y.x, f.x_out = y.x, f.width = W, f.top = l.spec.top, f.m = y.ex.m, f.w = l.experts_down.w, f.pitch = l.experts_down.pitch, f.rows_pad = l.expert_down_rows();
    f.chosen = y.ex.chosen, f.weight = y.ex.weight, f.shared_m = y.m, f.shared_w = l.down.w, f.shared_pitch = l.down.pitch, f.shared_scale = y.ex.shared_scale, f.depth = layered_depth(y, li);
    f.rows = std::min(kMoeDownRows, std::max(1, (W + 4 * m.sm_count - 1) / (4 * m.sm_count)));
    launch_dependent(moe_down_step_kernel<T>, dim3((W + f.rows - 1) / f.rows), kProjectThreads, (size_t(f.top) * f.pitch + f.shared_pitch) * sizeof(float), s, f);
    QTB_LAUNCH_CHECK();
    return QUINTRIT_OK;
}

// The chosen experts of n tokens whose normed inputs are in y.h2 and whose router logits are in y.ex.logits; results by pair row in y.ex.out.
template <typename T>
int layered_experts(quintrit_b200_decoder* d, size_t li, int n) {
    LayeredDecoder& y = *d->lay;
    const LayeredLayer& l = y.model->layers[li];
    const LayerSpec& sp = l.spec;
    LayeredDecoder::Experts& x = y.ex;
    cudaStream_t s = d->stream;
    MoeRouteArgs r{};
    r.router = layered_router(sp), r.tokens = n, r.logits = x.logits, r.chosen = x.chosen, r.weight = x.weight, r.count = x.count, r.rank = x.rank, r.first = x.first, r.row = x.row;
    r.up_runs = x.up_runs, r.down_runs = x.down_runs, r.n_runs = x.n_runs, r.up_rows = l.expert_rows(), r.down_rows = l.expert_down_rows(), r.tile = sizeof(T) != 2 ? kF32Tile : n * sp.top >= 160 * sp.experts ? 256 : 128;  // (the wider tile where an expert's share fills most of it)
    moe_route_kernel<<<(n + 3) / 4, 128, size_t(8) * sp.experts * sizeof(uint32_t), s>>>(r);
    QTB_LAUNCH_CHECK();
    moe_plan_kernel<<<1, 1024, 0, s>>>(r);
    QTB_LAUNCH_CHECK();
    moe_gather_kernel<<<dim3(sp.top, n), 128, 0, s>>>(r, static_cast<const uint4*>(y.h2), static_cast<uint4*>(x.h), static_cast<int>(l.experts_in.pitch * sizeof(T) / 16));
    QTB_LAUNCH_CHECK();
    auto grouped = [&](const LayeredMatrix& w, int rows, const CUtensorMap& map, const void* act, const DenseRun* runs, const DenseSeg& seg) -> int {
        DenseGemmArgs a{};
        a.tokens = n * sp.top, a.n_prob = 1, a.k_steps[0] = w.pitch / kDenseK, a.row_tiles[0] = rows / kDenseM, a.runs = runs, a.n_runs = x.n_runs;
        a.stack[0] = layered_stack(w), a.stack[0].n_seg = 1, a.stack[0].seg[0] = seg, a.status = d->d_counters + 2, a.spin_limit = kDenseSpinLimit;
        const int most = n * sp.top / r.tile + std::min(sp.experts, n * sp.top);  // runs there can be
        const int blocks = std::min(d->sm_count, most * a.row_tiles[0]);
        if constexpr (sizeof(T) == 2)
            r.tile == 256 ? dense_gemm_tc_kernel<256, kDenseGrouped><<<blocks, kDenseThreads, dense_smem(256), s>>>(w.map, map, w.map, map, a)
                          : dense_gemm_tc_kernel<128, kDenseGrouped><<<blocks, kDenseThreads, dense_smem(128), s>>>(w.map, map, w.map, map, a);
        else
            dense_gemm_f32_kernel<kDenseGrouped><<<dim3(most, a.row_tiles[0] * (kDenseM / kF32Tile)), 256, 0, s>>>(
                static_cast<const float*>(w.w), static_cast<const float*>(act), w.pitch, static_cast<const float*>(w.w), static_cast<const float*>(act), w.pitch, a);
        QTB_LAUNCH_CHECK();
        return QUINTRIT_OK;
    };
    const int W = y.model->spec.width;
    static const CUtensorMap no_map{};
    int rc = grouped(l.experts_in, l.expert_rows(), x.map_h, x.h, x.up_runs, DenseSeg{0, 2 * sp.ff, kSegSwiGlu, l.experts_down.pitch, nullptr, x.m, nullptr});
    if (rc != QUINTRIT_OK) return rc;
    return grouped(l.experts_down, l.expert_down_rows(), sizeof(T) == 2 ? x.map_m[li] : no_map, x.m, x.down_runs, DenseSeg{0, W, kSegStore, W, nullptr, x.out, nullptr});
}

// The same layer, many tokens: y.h1 holds the first norm's result when it begins (*normed; else it is made here) and the next layer's when it ends.
template <typename T>
int layered_sequential_layer(quintrit_b200_decoder* d, size_t li, int n, const LayeredTarget& tg, bool* normed) {
    LayeredDecoder& y = *d->lay;
    const LayeredModel& m = *y.model;
    const LayeredLayer& l = m.layers[li];
    cudaStream_t s = d->stream;
    const int W = m.spec.width, wp = m.embed.pitch, sets = static_cast<int>(l.mix.size());
    const bool experts = l.spec.ff_kind == FfKind::kExperts;
    int rc;
    DenseStack st[2] = {};
    layered_in_stacks(y, l, st);
    if (!*normed) {
        norm_rows_kernel<T><<<n, 256, 0, s>>>(y.x, W, m.spec.eps, l.norm1, static_cast<T*>(y.h1), NormParams{}, nullptr, wp, nullptr);
        QTB_LAUNCH_CHECK();
    }
    *normed = true;
    {
        const LayeredMatrix* const ws[2] = {&l.in1, &l.in1};
        const CUtensorMap* const hm[2] = {&y.map_h1, &y.map_h1};
        const void* const hs[2] = {y.h1, y.h1};
        if ((rc = layered_gemm<T>(d, n, ws, hm, hs, st, 1)) != QUINTRIT_OK) return rc;
    }
    for (int k = 0; k < sets; ++k) {
        const LayeredMixer& x = l.mix[k];
        bool ready;
        if ((rc = layered_mixer<T>(d, li, k, n, tg, &ready)) != QUINTRIT_OK) return rc;
        if (ready) continue;
        const float* gate = x.spec.kind == MixerKind::kRetention ? y.p1 + x.col + x.spec.gate_col() : nullptr;
        finish_rows_kernel<T><<<n, 256, size_t(x.spec.inner()) * sizeof(float), s>>>(y.y[k], nullptr, gate, l.spec.in_rows(), x.spec.inner(), layered_norm_parts(x.spec), m.spec.eps, nullptr, 1,
                                                                                     static_cast<T*>(y.y_t[k]), x.o.pitch);
        QTB_LAUNCH_CHECK();
    }
    RowsArgs r{};
    r.x = y.x, r.x_out = y.x, r.width = W, r.pitch = wp, r.eps = m.spec.eps;
    if (sets > 1) {
        const LayeredMatrix* const ws[2] = {&l.mix[0].o, &l.mix[1].o};
        const CUtensorMap* const hm[2] = {&y.map_y[l.mixer0], &y.map_y[l.mixer0 + 1]};
        const void* const hs[2] = {y.y_t[0], y.y_t[1]};
        DenseStack so[2] = {layered_stack(l.mix[0].o), layered_stack(l.mix[1].o)};
        so[0].n_seg = 1, so[0].seg[0] = DenseSeg{0, W, kSegPlain, W, y.g1, nullptr, nullptr};
        so[1].n_seg = 1, so[1].seg[0] = DenseSeg{0, W, kSegPlain, W, y.g2, nullptr, nullptr};
        if ((rc = layered_gemm<T>(d, n, ws, hm, hs, so, 2)) != QUINTRIT_OK) return rc;
        r.pair = PairSum{{y.g1, y.g2}, {l.mix[0].result_norm, l.mix[1].result_norm}};
    } else {
        DenseGemmArgs a{};
        a.x = y.x;
        if ((rc = layered_add<T>(d, n, &l.mix[0].o, &y.map_y[l.mixer0], y.y_t[0], nullptr, nullptr, nullptr, a)) != QUINTRIT_OK) return rc;
    }
    if (experts) {
        r.norm = l.norm2, r.h = y.h2;
        rows_kernel<T><<<n, 256, size_t(W) * sizeof(float), s>>>(r);
        QTB_LAUNCH_CHECK();
        const LayeredMatrix* const ws[2] = {&l.in2, &l.in2};
        const CUtensorMap* const hm[2] = {&y.map_h2, &y.map_h2};
        const void* const hs[2] = {y.h2, y.h2};
        DenseStack sr[2] = {st[1], {}};
        if ((rc = layered_gemm<T>(d, n, ws, hm, hs, sr, 1)) != QUINTRIT_OK || (rc = layered_experts<T>(d, li, n)) != QUINTRIT_OK) return rc;
        DenseGemmArgs a{};
        a.x = y.x, a.token_gate = y.ex.shared_scale;
        if ((rc = layered_add<T>(d, n, &l.down, &y.map_m[li], y.m, nullptr, nullptr, nullptr, a)) != QUINTRIT_OK) return rc;
        r.pair = PairSum{};
        r.pick = y.ex.out, r.pick_row = y.ex.row, r.pick_weight = y.ex.weight, r.top = l.spec.top;
    }
    r.depth = layered_depth(y, li);
    const bool more = li + 1 < m.layers.size();
    r.norm = more ? m.layers[li + 1].norm1 : NormParams{}, r.h = more ? y.h1 : nullptr;
    rows_kernel<T><<<n, 256, size_t(W) * sizeof(float), s>>>(r);
    QTB_LAUNCH_CHECK();
    return QUINTRIT_OK;
}

// Embedding and all layers for the n tokens in `tokens`; the residual stream ends in y.x.
template <typename T>
int layered_layers(quintrit_b200_decoder* d, const uint32_t* tokens, int n, const LayeredTarget& tg) {
    LayeredDecoder& y = *d->lay;
    const LayeredModel& m = *y.model;
    cudaStream_t s = d->stream;
    const int W = m.spec.width, wp = m.embed.pitch;
    if (m.embed_norm.w != nullptr)
        embed_norm_kernel<T><<<n, 256, size_t(W) * sizeof(float), s>>>(static_cast<const T*>(m.embed.w), wp, tokens, W, m.spec.eps, m.embed_norm, y.x, y.past, m.layers[0].norm1,
                                                                      static_cast<T*>(n > 1 ? y.h1 : nullptr));
    else
        embed_scaled_kernel<T><<<dim3((W + 255) / 256, n), 256, 0, s>>>(static_cast<const T*>(m.embed.w), wp, static_cast<const T*>(m.pos_table), tokens, tg.pos, tg.seq, m.spec.embed_scale, W, y.x);
    QTB_LAUNCH_CHECK();
    bool normed = m.embed_norm.w != nullptr;  // y.h1 holds the next layer's first norm
    for (size_t li = 0; li < m.layers.size(); ++li) {
        const bool parallel = m.layers[li].spec.parallel;
        const int rc = parallel ? layered_parallel_layer<T>(d, li, n, tg) : n == 1 ? layered_sequential_step<T>(d, li, tg) : layered_sequential_layer<T>(d, li, n, tg, &normed);
        if (rc != QUINTRIT_OK) return rc;
        if (parallel) normed = false;
    }
    return QUINTRIT_OK;
}

// Final norm and output table of one row of the residual stream -> d->logits.
template <typename T>
int layered_head(quintrit_b200_decoder* d, int row, float* logits) {
    LayeredDecoder& y = *d->lay;
    const LayeredModel& m = *y.model;
    NormProjectArgs a{};
    a.x = y.x + size_t(row) * m.spec.width, a.norm[0] = m.out_norm, a.eps = m.spec.eps, a.width = m.spec.width, a.n_stack = 1;
    a.stack[0] = layered_stack(m.head);
    a.stack[0].n_seg = 1, a.stack[0].seg[0] = DenseSeg{0, m.spec.vocab, kSegPlain, m.spec.vocab, logits, nullptr, nullptr};
    const int warps = kProjectThreads / 32;
    launch_dependent(layered_project_kernel<T>(a), dim3(std::min((m.spec.vocab / 2 + warps) / warps, 4 * m.sm_count)), kProjectThreads, size_t(m.head.pitch) * sizeof(float), d->stream, a);
    QTB_LAUNCH_CHECK();
    return QUINTRIT_OK;
}

// The same for n <= kDenseBox rows - those listed in `rows`, or first .. first + n - 1 where it is nullptr -> logits[n][vocab].
template <typename T>
int layered_head_rows(quintrit_b200_decoder* d, const uint32_t* rows, int first, int n, float* logits) {
    LayeredDecoder& y = *d->lay;
    const LayeredModel& m = *y.model;
    norm_rows_kernel<T><<<n, 256, 0, d->stream>>>(y.x + size_t(first) * m.spec.width, m.spec.width, m.spec.eps, m.out_norm, static_cast<T*>(y.h_head), NormParams{}, nullptr, m.head.pitch, rows);
    QTB_LAUNCH_CHECK();
    DenseStack st[2] = {layered_stack(m.head), {}};
    st[0].n_seg = 1, st[0].seg[0] = DenseSeg{0, m.spec.vocab, kSegPlain, m.spec.vocab, logits, nullptr, nullptr};
    const LayeredMatrix* const ws[2] = {&m.head, &m.head};
    const CUtensorMap* const hm[2] = {&y.map_head, &y.map_head};
    const void* const hs[2] = {y.h_head, y.h_head};
    return layered_gemm<T>(d, n, ws, hm, hs, st, 1);
}

// ---- what the decoder calls ---------------------------------------------------------------------------------------------------------------
inline LayeredTarget layered_own(quintrit_b200_decoder* d, const uint32_t* pos) {
    LayeredTarget t;
    t.store = &d->lay->store, t.pos = pos;
    return t;
}
inline int layered_run(quintrit_b200_decoder* d, const uint32_t* tokens, int n, const LayeredTarget& tg) {
    return d->lay->model->f32 ? layered_layers<float>(d, tokens, n, tg) : layered_layers<bf16>(d, tokens, n, tg);
}
inline int layered_logits(quintrit_b200_decoder* d, int row, float* logits) {
    return d->lay->model->f32 ? layered_head<float>(d, row, logits) : layered_head<bf16>(d, row, logits);
}
inline int layered_logits_rows(quintrit_b200_decoder* d, const uint32_t* rows, int n, float* logits) {
    return d->lay->model->f32 ? layered_head_rows<float>(d, rows, 0, n, logits) : layered_head_rows<bf16>(d, rows, 0, n, logits);
}
inline int layered_logits_rows(quintrit_b200_decoder* d, int first, int n, float* logits) {
    return d->lay->model->f32 ? layered_head_rows<float>(d, nullptr, first, n, logits) : layered_head_rows<bf16>(d, nullptr, first, n, logits);
}

// One token (id and position in device memory), logits and greedy choice: the body of the decoder's step graph.
int layered_enqueue_token(quintrit_b200_decoder* d, bool with_head) {
    int rc = layered_run(d, d->d_token, 1, layered_own(d, d->d_pos));
    if (rc != QUINTRIT_OK || !with_head) return rc;
    if ((rc = layered_logits(d, 0, d->logits)) != QUINTRIT_OK) return rc;
    argmax_kernel<<<1, 1024, 0, d->stream>>>(d->logits, d->vocab, d->d_token);
    QTB_LAUNCH_CHECK();
    return QUINTRIT_OK;
}

// Tokens at positions pos0 .. pos0 + count - 1 of a sequence, in chunks; logits at the places `want` (ascending indices into tokens) go to
// want_logits (host, [want_n][vocab]); the last token's logits and greedy choice are left in d->logits / d->d_token.
int layered_prefill(quintrit_b200_decoder* d, const uint32_t* tokens, size_t count, uint32_t pos0, const LayeredStore* store, int slot, const uint32_t* want, size_t want_n, float* want_logits) {
    LayeredDecoder& y = *d->lay;
    cudaStream_t s = d->stream;
    const bool own = store == nullptr;
    LayeredTarget tg = layered_own(d, y.pos);
    if (!own) tg.store = store, tg.slot = slot;
    int rc;
    if (want_n > 0 && y.many_logits == nullptr && (rc = dev_alloc(d, &y.many_logits, size_t(kLayeredLogitRows) * d->vocab, false)) != QUINTRIT_OK) return rc;
    size_t w0 = 0;
    for (size_t c0 = 0; c0 < count; c0 += kLayeredChunk) {
        const int n = static_cast<int>(std::min<size_t>(kLayeredChunk, count - c0));
        const uint32_t p = pos0 + static_cast<uint32_t>(c0);
        QTB_CUDA(cudaMemcpyAsync(y.tokens, tokens + c0, size_t(n) * sizeof(uint32_t), cudaMemcpyHostToDevice, s));
        QTB_CUDA(cudaMemcpyAsync(y.pos, &p, sizeof p, cudaMemcpyHostToDevice, s));
        if ((rc = layered_run(d, y.tokens, n, tg)) != QUINTRIT_OK) return rc;
        while (w0 < want_n && want[w0] < c0 + n) {
            std::vector<uint32_t> rows;
            for (size_t i = w0; i < want_n && want[i] < c0 + n && rows.size() < size_t(kLayeredLogitRows); ++i) rows.push_back(want[i] - static_cast<uint32_t>(c0));
            QTB_CUDA(cudaMemcpyAsync(y.rows, rows.data(), rows.size() * sizeof(uint32_t), cudaMemcpyHostToDevice, s));
            if ((rc = layered_logits_rows(d, y.rows, static_cast<int>(rows.size()), y.many_logits)) != QUINTRIT_OK) return rc;
            QTB_CUDA(cudaMemcpyAsync(want_logits + w0 * d->vocab, y.many_logits, rows.size() * d->vocab * sizeof(float), cudaMemcpyDeviceToHost, s));
            QTB_CUDA(cudaStreamSynchronize(s));  // (the row list is a local of this turn)
            w0 += rows.size();
        }
        if (c0 + n < count) continue;
        if ((rc = layered_logits(d, n - 1, d->logits)) != QUINTRIT_OK) return rc;
        argmax_kernel<<<1, 1024, 0, s>>>(d->logits, d->vocab, d->d_token);
        QTB_LAUNCH_CHECK();
    }
    if (own) {  // position and history as after `count` single steps
        const uint32_t next = pos0 + static_cast<uint32_t>(count);
        QTB_CUDA(cudaMemcpyAsync(d->d_pos, &next, sizeof next, cudaMemcpyHostToDevice, s));
        QTB_CUDA(cudaMemcpyAsync(d->d_history + next - 1, d->d_token, sizeof(uint32_t), cudaMemcpyDeviceToDevice, s));
    }
    return QUINTRIT_OK;
}

// Timing a step must not change the sequence: the recurrent state is copied away before and back after (cache entries at a free position
// are overwritten by the next real token).
int layered_save(quintrit_b200_decoder* d, bool restore) {
    LayeredDecoder& y = *d->lay;
    const size_t bytes = y.store.recurrent_floats * sizeof(float);
    if (bytes == 0) return QUINTRIT_OK;
    if (y.recurrent_backup == nullptr)
        if (int rc = dev_alloc(d, &y.recurrent_backup, y.store.recurrent_floats, false)) return rc;
    QTB_CUDA(cudaMemcpyAsync(restore ? y.store.recurrent : y.recurrent_backup, restore ? y.recurrent_backup : y.store.recurrent, bytes, cudaMemcpyDeviceToDevice, d->stream));
    return QUINTRIT_OK;
}

// A position a sequence that holds `cached` tokens may continue from.
int layered_check_position(const quintrit_b200_decoder* d, uint32_t pos, uint32_t cached) {
    if (pos == cached || pos == 0) return QUINTRIT_OK;
    return fail(QUINTRIT_ERR_UNSUPPORTED, "position %u: this model's layers keep a state of all %u tokens; a sequence continues from its end or starts again from position 0", pos, cached);
}

// A decoder (sequence store, buffers) over loaded weights.
int layered_decoder_create(const std::shared_ptr<LayeredModel>& model, uint32_t ctx, quintrit_b200_decoder** out) {
    const LayeredModel& m = *model;
    quintrit_b200_decoder* d = new quintrit_b200_decoder();
    *out = d;  // the caller destroys it on failure
    d->magic = kMagicDecoder;
    d->device = m.device, d->sm_count = m.sm_count, d->arch = QUINTRIT_B200_ARCH_LAYERED, d->f32_values = 1;
    d->hidden = m.spec.width, d->layers = static_cast<int>(m.layers.size());
    for (const LayeredLayer& l : m.layers) {
        d->inter = std::max(d->inter, l.spec.ff);
        for (const LayeredMixer& x : l.mix)
            if (x.spec.cached() && d->q_heads == 0) d->q_heads = x.spec.heads, d->kv_heads = x.spec.kv_heads, d->head_dim = x.spec.dim;
    }
    d->vocab = d->vocab_full = m.spec.vocab, d->ctx = static_cast<int>(ctx), d->eps = m.spec.eps;
    d->bf16_tables = !m.f32;
    int rc;
    QTB_CUDA(cudaStreamCreateWithFlags(&d->stream, cudaStreamNonBlocking));
    if ((rc = dev_alloc(d, &d->logits, d->vocab)) || (rc = dev_alloc(d, &d->d_token, 4)) || (rc = dev_alloc(d, &d->d_pos, 4)) || (rc = dev_alloc(d, &d->d_history, size_t(ctx) + 1)) ||
        (rc = dev_alloc(d, &d->d_counters, 4)))
        return rc;
    return layered_decoder_setup(d, model);
}

}  // namespace qtb
