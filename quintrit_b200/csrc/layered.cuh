// Decoder of a layered model (layered_spec.hpp) on the device: weights, sequence store, and the launch sequences of a decode step, a
// prompt chunk and a step of several sequences. It stands behind the same decoder handle as the ternary models: token, position, history
// and logits are the decoder's own (decoder.cuh), and so are its CUDA graph, greedy choice, sampling, sessions and batches.
//
// A decode step takes three launches a layer: norms and every projection of their results (norm_project_kernel), the mixer, and output
// norm + output and down projection + gates + residual sum (finish_project_kernel). Many tokens take the tensor cores: norms, one grouped
// product of both stacks, the mixer, its output norm, and one product of two accumulators that ends in the residual sum.
//
// Weights are stored in the serving type (bf16, or float when the model was opened in 32-bit mode). Rows of a stack start at multiples of
// 128 and columns are padded to 64, so that one layout serves the streaming kernels and the tensor cores.
#pragma once
#include <memory>

#include "chunk_scan.cuh"
#include "dense_gemm_tc.cuh"
#include "dense_gemv.cuh"
#include "gated_scan.cuh"
#include "layered_spec.hpp"
#include "pooled_attention.cuh"
#include "pooled_attention_mma.cuh"
#include "tensor_map.cuh"

namespace qtb {

constexpr int kLayeredChunk = 2048;     // tokens of a prompt chunk
constexpr int kLayeredLogitRows = 64;   // rows of logits computed at a time when several positions of a chunk are asked for
constexpr int kLayeredMaxBatch = 256;   // sequences of a batched step

inline int round_up(int v, int m) { return (v + m - 1) / m * m; }

struct LayeredMatrix {
    void* w = nullptr;
    int rows_pad = 0, pitch = 0, cols = 0;
    CUtensorMap map{};
};
struct LayeredLayer {
    LayerSpec spec;
    LayeredMatrix in1, in2, o, down;    // mixer projections + gate 1; gate | up interleaved + gate 2; output; down
    int gate1_row = 0, gate2_row = 0;   // first rows of the gates in their stacks
    float *norm1 = nullptr, *norm2 = nullptr, *gate1_bias = nullptr, *gate2_bias = nullptr;
    float *conv_w = nullptr, *conv_b = nullptr, *dt_bias = nullptr, *a_log = nullptr, *d_skip = nullptr, *mix_norm = nullptr, *f_bias = nullptr, *lower = nullptr;
};
// The weights on the device, shared by every decoder of the model.
struct LayeredModel {
    LayeredSpec spec;
    bool f32 = false;
    int device = 0, sm_count = 0;
    std::vector<LayeredLayer> layers;
    LayeredMatrix embed, head;
    void* pos_table = nullptr;
    float* out_norm = nullptr;
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
            if (l.spec.kind != MixerKind::kAttention) return true;
        return false;
    }
};

// What `slots` sequences hold: recurrent states (one allocation, so that a step can be timed and undone) and windowed caches.
struct LayeredStore {
    int slots = 0;
    float* recurrent = nullptr;
    size_t recurrent_floats = 0;
    struct Layer {
        float *state = nullptr, *conv = nullptr;
        size_t state_stride = 0, conv_stride = 0;  // floats per slot
        PooledCache cache{};
    };
    std::vector<Layer> layers;
};

struct LayeredDecoder {
    std::shared_ptr<LayeredModel> model;
    LayeredStore store;
    float* recurrent_backup = nullptr;
    uint32_t *tokens = nullptr, *pos = nullptr, *rows = nullptr;
    float *x = nullptr, *p1 = nullptr, *g1 = nullptr, *g2 = nullptr, *y = nullptr, *many_logits = nullptr;
    void *h1 = nullptr, *h2 = nullptr, *y_t = nullptr, *m = nullptr, *h_head = nullptr;
    CUtensorMap map_h1{}, map_h2{}, map_head{};
    std::vector<CUtensorMap> map_y, map_m;  // per layer: the pitches differ
    float *part_acc = nullptr, *part_ml = nullptr;
    unsigned int* done = nullptr;
    char* work = nullptr;               // chunked recurrences: operands of one layer (ChunkWork)
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
            d.spec = l;
            if (int rc = layer(l, &d)) return rc;
        }
        if (int rc = matrix({Part{{s.embed}, s.vocab}}, s.width, &m_->embed, nullptr)) return rc;
        if (s.head == s.embed) m_->head = m_->embed;
        else if (int rc = matrix({Part{{s.head}, s.vocab}}, s.width, &m_->head, nullptr)) return rc;
        if (!s.pos.empty())
            if (int rc = table(s.pos, {uint64_t(s.max_positions), uint64_t(s.width)}, &m_->pos_table)) return rc;
        if (int rc = floats(s.out_norm, {uint64_t(s.width)}, &m_->out_norm)) return rc;
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
    // Stacks the parts row-wise, each part padded to kRowPad rows; first_row (optional) receives the first row of the last part.
    int matrix(const std::vector<Part>& parts, int cols, LayeredMatrix* out, int* first_row) {
        int rows = 0;
        for (const Part& p : parts) rows += round_up(p.rows, kRowPad);
        out->rows_pad = rows, out->pitch = round_up(cols, kColPad), out->cols = cols;
        const size_t pitch = size_t(out->pitch) * m_->elem();
        stage_.assign(size_t(rows) * pitch, 0);
        int r0 = 0;
        for (const Part& p : parts) {
            if (first_row != nullptr) *first_row = r0;
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
    int layer(const LayerSpec& l, LayeredLayer* d) {
        const int W = m_->spec.width;
        const uint64_t w = W, inner = l.inner();
        std::vector<Part> p1{Part{l.in, l.in_rows()}};
        if (l.gated_residual) p1.push_back(Part{{l.gate1}, W});
        if (int rc = matrix(p1, W, &d->in1, &d->gate1_row)) return rc;
        if (int rc = matrix({Part{{l.out}, W}}, l.inner(), &d->o, nullptr)) return rc;
        if (int rc = floats(l.norm1, {w}, &d->norm1)) return rc;
        if (l.gated_residual)
            if (int rc = floats(l.gate1_bias, {w}, &d->gate1_bias)) return rc;
        if (l.ff > 0) {
            std::vector<Part> p2{Part{{l.ff_gate, l.ff_up}, 2 * l.ff, true}};
            if (l.gated_residual) p2.push_back(Part{{l.gate2}, W});
            if (int rc = matrix(p2, W, &d->in2, &d->gate2_row)) return rc;
            if (int rc = matrix({Part{{l.ff_down}, W}}, l.ff, &d->down, nullptr)) return rc;
            if (int rc = floats(l.norm2, {w}, &d->norm2)) return rc;
            if (l.gated_residual)
                if (int rc = floats(l.gate2_bias, {w}, &d->gate2_bias)) return rc;
        }
        const uint64_t heads = l.heads;
        int rc = QUINTRIT_OK;
        if (l.kind == MixerKind::kMamba2) {
            const uint64_t ch = l.conv_dim();
            (rc = floats(l.conv_w, {ch, uint64_t(l.conv)}, &d->conv_w)) || (rc = floats(l.conv_b, {ch}, &d->conv_b)) || (rc = floats(l.dt_bias, {heads}, &d->dt_bias)) ||
                (rc = floats(l.a_log, {heads}, &d->a_log)) || (rc = floats(l.d_skip, {heads}, &d->d_skip)) || (rc = floats(l.mix_norm, {inner}, &d->mix_norm));
        } else if (l.kind == MixerKind::kHgrn2) {
            const uint64_t hd = heads * l.dim;
            (rc = floats(l.f_bias, {hd}, &d->f_bias)) || (rc = floats(l.lower, {hd}, &d->lower)) || (rc = floats(l.mix_norm, {uint64_t(l.vdim)}, &d->mix_norm));
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
    st->layers.resize(m.layers.size());
    size_t total = 0;
    for (size_t i = 0; i < m.layers.size(); ++i) {
        const LayerSpec& l = m.layers[i].spec;
        LayeredStore::Layer& s = st->layers[i];
        if (l.kind == MixerKind::kAttention) continue;
        s.state_stride = size_t(l.heads) * l.vdim * l.key_dim();
        if (l.kind == MixerKind::kMamba2) s.conv_stride = size_t(l.conv) * l.conv_dim();
        total += (s.state_stride + s.conv_stride) * slots;
    }
    int rc = alloc(reinterpret_cast<void**>(&st->recurrent), std::max<size_t>(total, 4) * sizeof(float));
    if (rc != QUINTRIT_OK) return rc;
    st->recurrent_floats = total;
    float* p = st->recurrent;
    for (size_t i = 0; i < m.layers.size(); ++i) {
        const LayerSpec& l = m.layers[i].spec;
        LayeredStore::Layer& s = st->layers[i];
        if (l.kind != MixerKind::kAttention) {
            s.state = p, p += s.state_stride * slots;
            s.conv = p, p += s.conv_stride * slots;
            continue;
        }
        PooledCache& c = s.cache;
        c.ring = std::min(ctx, std::max(l.window, l.pool) + kLayeredChunk);
        c.blocks = l.pool > 0 ? ctx / l.pool + 1 : 0;
        const size_t dp = round_up(l.dim, 8), vp = round_up(l.vdim, 8), rows = size_t(slots) * c.ring * l.kv_heads, pools = size_t(slots) * c.blocks * l.kv_heads;
        if ((rc = alloc(&c.k, rows * dp * m.elem())) || (rc = alloc(&c.v, rows * vp * m.elem())) || (rc = alloc(&c.pk, pools * dp * m.elem())) || (rc = alloc(&c.pv, pools * vp * m.elem())))
            return rc;
    }
    return QUINTRIT_OK;
}

inline void layered_store_view(const LayeredModel& m, const LayeredStore& st, size_t layer, int slot, LayeredStore::Layer* out) {
    *out = st.layers[layer];
    if (slot == 0) return;
    const LayerSpec& l = m.layers[layer].spec;
    if (l.kind != MixerKind::kAttention) {
        out->state += out->state_stride * slot, out->conv += out->conv_stride * slot;
        return;
    }
    PooledCache& c = out->cache;
    const size_t dp = round_up(l.dim, 8) * m.elem(), vp = round_up(l.vdim, 8) * m.elem(), rows = size_t(slot) * c.ring * l.kv_heads, pools = size_t(slot) * c.blocks * l.kv_heads;
    c.k = static_cast<char*>(c.k) + rows * dp, c.v = static_cast<char*>(c.v) + rows * vp;
    c.pk = static_cast<char*>(c.pk) + pools * dp, c.pv = static_cast<char*>(c.pv) + pools * vp;
}

// Shares a decode step's attention is cut into: enough blocks for the device, none below one tile of keys.
inline int pooled_splits(const LayerSpec& l, int ctx, int n, int sm_count) {
    const int groups = l.kv_heads * ((l.heads / l.kv_heads + kPaHeads - 1) / kPaHeads) * n;
    const int keys = std::min(ctx, l.window) + (l.pool > 0 ? ctx / l.pool : 0);
    return std::max(1, std::min({(keys + kPaTile - 1) / kPaTile, 4 * sm_count / groups, 64}));
}

inline int layered_decoder_setup(quintrit_b200_decoder* d, const std::shared_ptr<LayeredModel>& model) {
    const LayeredModel& m = *model;
    LayeredDecoder* y = d->lay = new LayeredDecoder();
    y->model = model;
    auto alloc = [&](void** p, size_t bytes) { return dev_alloc(d, reinterpret_cast<char**>(p), bytes); };
    int rc = layered_store_create(m, 1, d->ctx, alloc, &y->store);
    if (rc != QUINTRIT_OK) return rc;
    const size_t C = kLayeredChunk, W = m.spec.width, wp = m.embed.pitch, e = m.elem();
    size_t work = 0, p1 = 0, inner = 0, op = 0, mp = kColPad, parts = 1, groups = 1, acc = 4;
    for (const LayeredLayer& l : m.layers) {
        p1 = std::max<size_t>(p1, l.spec.in_rows()), inner = std::max<size_t>(inner, l.spec.inner()), op = std::max<size_t>(op, l.o.pitch), mp = std::max<size_t>(mp, l.down.pitch);
        if (l.spec.kind != MixerKind::kAttention) {
            ChunkWork cw;
            if (!m.f32 && chunk_scan_rows(l.spec.key_dim()) != 0)
                work = std::max(work, chunk_work(nullptr, l.spec.kind == MixerKind::kMamba2, l.spec.heads, l.spec.vdim, l.spec.key_dim(), l.spec.groups, kLayeredChunk, &cw));
            continue;
        }
        groups = std::max<size_t>(groups, size_t(l.spec.kv_heads) * ((l.spec.heads / l.spec.kv_heads + kPaHeads - 1) / kPaHeads));
        for (int n = 1; n <= kLayeredMaxBatch; ++n) {
            const size_t sp = pooled_splits(l.spec, d->ctx, n, m.sm_count);
            if (sp > 1) parts = std::max(parts, n * l.spec.heads * sp), acc = std::max(acc, n * l.spec.heads * sp * l.spec.vdim);
        }
    }
    if ((rc = dev_alloc(d, &y->tokens, C)) || (rc = dev_alloc(d, &y->pos, 4)) || (rc = dev_alloc(d, &y->rows, C)) || (rc = dev_alloc(d, &y->x, C * W)) || (rc = dev_alloc(d, &y->p1, C * p1)) ||
        (rc = dev_alloc(d, &y->g1, C * W)) || (rc = dev_alloc(d, &y->g2, C * W)) || (rc = dev_alloc(d, &y->y, C * inner)) || (rc = alloc(&y->h1, C * wp * e)) ||
        (rc = alloc(&y->h2, C * wp * e)) || (rc = alloc(&y->y_t, C * op * e)) || (rc = alloc(&y->m, C * mp * e)) || (rc = alloc(&y->h_head, size_t(kDenseBox) * wp * e)) ||
        (rc = dev_alloc(d, &y->part_acc, acc)) || (rc = dev_alloc(d, &y->part_ml, 2 * parts)) || (rc = dev_alloc(d, &y->done, groups * kLayeredMaxBatch)) ||
        (rc = dev_alloc(d, &y->work, work)))
        return rc;
    if (!m.f32) {
        if ((rc = tensor_map_2d_bf16(&y->map_h1, y->h1, m.embed.pitch, C, kDenseK, kDenseBox)) || (rc = tensor_map_2d_bf16(&y->map_h2, y->h2, m.embed.pitch, C, kDenseK, kDenseBox)) ||
            (rc = tensor_map_2d_bf16(&y->map_head, y->h_head, m.embed.pitch, kDenseBox, kDenseK, kDenseBox)))
            return rc;
        y->map_y.resize(m.layers.size()), y->map_m.resize(m.layers.size());
        for (size_t i = 0; i < m.layers.size(); ++i) {
            if ((rc = tensor_map_2d_bf16(&y->map_y[i], y->y_t, m.layers[i].o.pitch, C, kDenseK, kDenseBox))) return rc;
            y->map_m[i] = y->map_y[i];
            if (m.layers[i].spec.ff > 0 && (rc = tensor_map_2d_bf16(&y->map_m[i], y->m, m.layers[i].down.pitch, C, kDenseK, kDenseBox))) return rc;
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
    const void* kernels[] = {reinterpret_cast<const void*>(norm_project_kernel<bf16>), reinterpret_cast<const void*>(norm_project_kernel<float>),
                             reinterpret_cast<const void*>(finish_project_kernel<bf16>), reinterpret_cast<const void*>(finish_project_kernel<float>),
                             reinterpret_cast<const void*>(finish_rows_kernel<bf16>), reinterpret_cast<const void*>(finish_rows_kernel<float>),
                             reinterpret_cast<const void*>(gated_scan_kernel<kScanMamba2>), reinterpret_cast<const void*>(gated_scan_kernel<kScanHgrn2>),
                             reinterpret_cast<const void*>(pooled_attention_kernel<bf16, true>), reinterpret_cast<const void*>(pooled_attention_kernel<bf16, false>),
                             reinterpret_cast<const void*>(pooled_attention_kernel<float, true>), reinterpret_cast<const void*>(pooled_attention_kernel<float, false>),
                             reinterpret_cast<const void*>(dense_gemm_tc_kernel<128, true>), reinterpret_cast<const void*>(dense_gemm_tc_kernel<128, false>),
                             reinterpret_cast<const void*>(dense_gemm_tc_kernel<256, false>),
                             reinterpret_cast<const void*>(chunk_scan_kernel<kScanMamba2, 32>), reinterpret_cast<const void*>(chunk_scan_kernel<kScanMamba2, 64>),
                             reinterpret_cast<const void*>(chunk_scan_kernel<kScanMamba2, 128>), reinterpret_cast<const void*>(chunk_scan_kernel<kScanHgrn2, 32>),
                             reinterpret_cast<const void*>(chunk_scan_kernel<kScanHgrn2, 64>), reinterpret_cast<const void*>(chunk_scan_kernel<kScanHgrn2, 128>),
                             reinterpret_cast<const void*>(pooled_attention_mma_kernel<32>), reinterpret_cast<const void*>(pooled_attention_mma_kernel<64>),
                             reinterpret_cast<const void*>(pooled_attention_mma_kernel<128>)};
    for (const void* k : kernels)
        if ((rc = allow(k)) != QUINTRIT_OK) return rc;
    // the largest requests of this model against what a block may have
    const size_t limit = static_cast<size_t>(optin) - 2048;
    for (const LayeredLayer& l : m.layers) {
        size_t need = std::max<size_t>({2 * wp * 4, (size_t(l.o.pitch) + l.down.pitch) * 4, size_t(l.spec.inner()) * 4});
        if (l.spec.kind == MixerKind::kAttention) need = std::max(need, pooled_attn_smem(round_up(l.spec.dim, 8), round_up(l.spec.vdim, 8), static_cast<int>(e)));
        else need = std::max(need, scan_smem(l.spec.key_dim()));
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

// The two stacks of a layer's projections with their endings; returns how many there are.
inline int layered_in_stacks(const LayeredDecoder& y, const LayeredLayer& l, DenseStack (&st)[2]) {
    const int W = y.model->spec.width, rows = l.spec.in_rows();
    st[0] = layered_stack(l.in1);
    st[0].seg[st[0].n_seg++] = DenseSeg{0, rows, kSegPlain, rows, y.p1, nullptr, nullptr};
    if (l.spec.gated_residual) st[0].seg[st[0].n_seg++] = DenseSeg{l.gate1_row, W, kSegSigmoid, W, y.g1, nullptr, l.gate1_bias};
    if (l.spec.ff == 0) return 1;
    st[1] = layered_stack(l.in2);
    st[1].seg[st[1].n_seg++] = DenseSeg{0, 2 * l.spec.ff, kSegSwiGlu, l.down.pitch, nullptr, y.m, nullptr};
    if (l.spec.gated_residual) st[1].seg[st[1].n_seg++] = DenseSeg{l.gate2_row, W, kSegSigmoid, W, y.g2, nullptr, l.gate2_bias};
    return 2;
}

inline int layered_norm_parts(const LayerSpec& l) { return l.kind == MixerKind::kMamba2 ? l.norm_groups : l.kind == MixerKind::kHgrn2 ? l.heads : 0; }
inline int layered_norm_len(const LayerSpec& l) { return l.kind == MixerKind::kMamba2 ? l.inner() : l.vdim; }

// Many tokens of a recurrence in 16-token chunks.
inline int layered_chunk_scan(quintrit_b200_decoder* d, const LayerSpec& l, const ScanArgs& a) {
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

template <typename T>
int layered_mixer(quintrit_b200_decoder* d, size_t li, int n, const LayeredTarget& tg) {
    LayeredDecoder& y = *d->lay;
    const LayerSpec& l = y.model->layers[li].spec;
    const LayeredLayer& w = y.model->layers[li];
    cudaStream_t s = d->stream;
    LayeredStore::Layer st;
    layered_store_view(*y.model, *tg.store, li, tg.slot, &st);
    const int tokens = tg.step() ? 1 : n, seqs = tg.step() ? n : 1;
    if (l.kind != MixerKind::kAttention) {
        ScanArgs a{};
        a.tokens = tokens, a.pos = tg.pos, a.seq = tg.seq, a.p = y.p1, a.ld = l.in_rows();
        a.heads = l.heads, a.vdim = l.vdim, a.n = l.key_dim(), a.groups = l.groups, a.taps = l.conv;
        a.conv_w = w.conv_w, a.conv_b = w.conv_b, a.dt_bias = w.dt_bias, a.a_log = w.a_log, a.d_skip = w.d_skip, a.f_bias = w.f_bias, a.lower = w.lower;
        a.state = st.state, a.conv = st.conv, a.y = y.y;
        const dim3 grid(l.heads, (l.vdim + kScanRows - 1) / kScanRows, seqs);
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
    PooledAttnArgs a{};
    a.tokens = tokens, a.pos = tg.pos, a.seq = tg.seq, a.p = y.p1, a.ld = l.in_rows();
    a.heads = l.heads, a.kv_heads = l.kv_heads, a.dim = l.dim, a.vdim = l.vdim, a.dim_pad = round_up(l.dim, 8), a.vdim_pad = round_up(l.vdim, 8);
    a.window = l.window, a.pool = l.pool, a.scale = l.scale, a.head_gate = l.head_gate, a.cache = st.cache, a.y = y.y;
    a.part_acc = y.part_acc, a.part_ml = y.part_ml, a.done = y.done;
    const int hg = l.kv_heads * ((l.heads / l.kv_heads + kPaHeads - 1) / kPaHeads);
    const size_t smem = pooled_attn_smem(a.dim_pad, a.vdim_pad, sizeof(T));
    if (tokens == 1) {  // a token at a time: the attention kernel appends to the cache itself
        a.splits = pooled_splits(l, d->ctx, n, y.model->sm_count);
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

constexpr unsigned int kDenseSpinLimit = 1u << 16;  // polls of up to 20 us each: about a second before a wait gives up

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
            dense_gemm_tc_kernel<256, false><<<std::min(d->sm_count, (n + 255) / 256 * tiles), kDenseThreads, dense_smem(256), d->stream>>>(w[0]->map, *hmap[0], w[j]->map, *hmap[j], a);
        else
            dense_gemm_tc_kernel<128, false><<<std::min(d->sm_count, tiles), kDenseThreads, dense_smem(128), d->stream>>>(w[0]->map, *hmap[0], w[j]->map, *hmap[j], a);
    else
        dense_gemm_f32_kernel<false><<<dim3((n + kF32Tile - 1) / kF32Tile, tiles * (kDenseM / kF32Tile)), 256, 0, d->stream>>>(
            static_cast<const float*>(w[0]->w), static_cast<const float*>(h[0]), w[0]->pitch, static_cast<const float*>(w[j]->w), static_cast<const float*>(h[j]), w[j]->pitch, a);
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
    int rc;
    embed_scaled_kernel<T><<<dim3((W + 255) / 256, n), 256, 0, s>>>(static_cast<const T*>(m.embed.w), wp, static_cast<const T*>(m.pos_table), tokens, tg.pos, tg.seq, m.spec.embed_scale, W, y.x);
    QTB_LAUNCH_CHECK();
    for (size_t li = 0; li < m.layers.size(); ++li) {
        const LayeredLayer& l = m.layers[li];
        DenseStack st[2] = {};
        const int n_stack = layered_in_stacks(y, l, st);
        const int parts = layered_norm_parts(l.spec), norm_len = layered_norm_len(l.spec);
        if (n == 1) {
            NormProjectArgs a{};
            a.x = y.x, a.norm_w[0] = l.norm1, a.norm_w[1] = l.norm2, a.eps = m.spec.eps, a.width = W, a.n_stack = n_stack;
            int units = 0;
            for (int i = 0; i < n_stack; ++i) {
                a.stack[i] = st[i];
                for (int k = 0; k < st[i].n_seg; ++k) units += (st[i].seg[k].rows + 1) / 2;
            }
            const int warps = kProjectThreads / 32;
            launch_dependent(norm_project_kernel<T>, dim3(std::min((units + warps - 1) / warps, 4 * m.sm_count)), kProjectThreads, size_t(n_stack) * wp * sizeof(float), s, a);
            QTB_LAUNCH_CHECK();
            if ((rc = layered_mixer<T>(d, li, n, tg)) != QUINTRIT_OK) return rc;
            FinishProjectArgs f{};
            f.x = y.x, f.width = W, f.y = y.y, f.inner = l.spec.inner(), f.norm_parts = parts, f.norm_len = norm_len, f.norm_w = l.mix_norm, f.eps = m.spec.eps;
            f.o = l.o.w, f.o_pitch = l.o.pitch;
            if (l.spec.ff > 0) f.m = y.m, f.down = l.down.w, f.down_pitch = l.down.pitch;
            if (l.spec.gated_residual) f.gate1 = y.g1, f.gate2 = y.g2;
            launch_dependent(finish_project_kernel<T>, dim3(std::min((W + warps - 1) / warps, 4 * m.sm_count)), kProjectThreads, (size_t(f.o_pitch) + f.down_pitch) * sizeof(float), s, f);
            QTB_LAUNCH_CHECK();
            continue;
        }
        norm_rows_kernel<T><<<n, 256, 0, s>>>(y.x, W, m.spec.eps, l.norm1, static_cast<T*>(y.h1), l.norm2, n_stack > 1 ? static_cast<T*>(y.h2) : nullptr, wp, nullptr);
        QTB_LAUNCH_CHECK();
        const LayeredMatrix* const ws[2] = {&l.in1, &l.in2};
        const CUtensorMap* const hm[2] = {&y.map_h1, &y.map_h2};
        const void* const hs[2] = {y.h1, y.h2};
        if ((rc = layered_gemm<T>(d, n, ws, hm, hs, st, n_stack)) != QUINTRIT_OK || (rc = layered_mixer<T>(d, li, n, tg)) != QUINTRIT_OK) return rc;
        const float* gate = sizeof(T) == 2 && l.spec.kind == MixerKind::kMamba2 && !tg.step() && n > kChunkT / 2 && chunk_scan_rows(l.spec.state) != 0 ? y.p1 : nullptr;  // silu(z)
        finish_rows_kernel<T><<<n, 256, size_t(l.spec.inner()) * sizeof(float), s>>>(y.y, gate, l.spec.in_rows(), l.spec.inner(), parts, m.spec.eps, l.mix_norm, norm_len, static_cast<T*>(y.y_t), l.o.pitch);
        QTB_LAUNCH_CHECK();
        DenseGemmArgs a{};
        a.tokens = n, a.n_prob = 1, a.status = d->d_counters + 2, a.spin_limit = kDenseSpinLimit;
        a.k_steps[0] = l.o.pitch / kDenseK, a.k_steps[1] = l.spec.ff > 0 ? l.down.pitch / kDenseK : 0, a.row_tiles[0] = l.o.rows_pad / kDenseM;
        a.x = y.x, a.width = W;
        if (l.spec.gated_residual) a.gate1 = y.g1, a.gate2 = y.g2;
        if constexpr (sizeof(T) == 2)
            dense_gemm_tc_kernel<128, true><<<std::min(d->sm_count, (n + 127) / 128 * a.row_tiles[0]), kDenseThreads, dense_smem(128), s>>>(l.o.map, y.map_y[li], l.spec.ff > 0 ? l.down.map : l.o.map, y.map_m[li], a);
        else
            dense_gemm_f32_kernel<true><<<dim3((n + kF32Tile - 1) / kF32Tile, a.row_tiles[0] * (kDenseM / kF32Tile)), 256, 0, s>>>(
                static_cast<const float*>(l.o.w), static_cast<const float*>(y.y_t), l.o.pitch, static_cast<const float*>(l.down.w), static_cast<const float*>(y.m), l.down.pitch, a);
        QTB_LAUNCH_CHECK();
    }
    return QUINTRIT_OK;
}

// Final norm and output table of one row of the residual stream -> d->logits.
template <typename T>
int layered_head(quintrit_b200_decoder* d, int row, float* logits) {
    LayeredDecoder& y = *d->lay;
    const LayeredModel& m = *y.model;
    NormProjectArgs a{};
    a.x = y.x + size_t(row) * m.spec.width, a.norm_w[0] = m.out_norm, a.eps = m.spec.eps, a.width = m.spec.width, a.n_stack = 1;
    a.stack[0] = layered_stack(m.head);
    a.stack[0].n_seg = 1, a.stack[0].seg[0] = DenseSeg{0, m.spec.vocab, kSegPlain, m.spec.vocab, logits, nullptr, nullptr};
    const int warps = kProjectThreads / 32;
    launch_dependent(norm_project_kernel<T>, dim3(std::min((m.spec.vocab / 2 + warps) / warps, 4 * m.sm_count)), kProjectThreads, size_t(m.head.pitch) * sizeof(float), d->stream, a);
    QTB_LAUNCH_CHECK();
    return QUINTRIT_OK;
}

// The same for n <= kDenseBox rows - those listed in `rows`, or first .. first + n - 1 where it is nullptr -> logits[n][vocab].
template <typename T>
int layered_head_rows(quintrit_b200_decoder* d, const uint32_t* rows, int first, int n, float* logits) {
    LayeredDecoder& y = *d->lay;
    const LayeredModel& m = *y.model;
    norm_rows_kernel<T><<<n, 256, 0, d->stream>>>(y.x + size_t(first) * m.spec.width, m.spec.width, m.spec.eps, m.out_norm, static_cast<T*>(y.h_head), nullptr, nullptr, m.head.pitch, rows);
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
        if (l.spec.kind == MixerKind::kAttention && d->q_heads == 0) d->q_heads = l.spec.heads, d->kv_heads = l.spec.kv_heads, d->head_dim = l.spec.dim;
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
