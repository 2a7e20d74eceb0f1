// Attention whose weights are not normalized over the keys: position i gives every earlier key j the weight
//
//   sigmoid(scale q . k - slope_h (i - j) + bias_h)
//
// and adds the weighted values up. Before that, queries and keys are RMS-normed over a token's whole projection (all heads at once), queries are
// multiplied by a temperature that grows with the position, and each head's value is divided by its root mean square. Keys and values are
// cached as they are used, in the storage type; norms, scores and weights are 32-bit.
//
// The cache of a layer and sequence holds `capacity` rows of [kv head][dim padded to 8]; position p lies in row p.
#pragma once
#include "mma_bf16.cuh"
#include "pooled_attention_mma.cuh"

namespace qtb {

struct LogisticArgs {
    int tokens;               // consecutive tokens of a sequence (1 per sequence in a step)
    const uint32_t* pos;
    SeqIndex seq;
    const float* p;           // projections [token][ld]: q | k | v
    int ld;
    int heads, kv_heads, dim, vdim, dim_pad, vdim_pad;
    float scale, eps;
    const float *q_norm, *k_norm;   // weights over heads * dim and kv_heads * dim; nullptr: no norm
    float temp_coef, temp_every;    // q times 1 + coef ln(floor((pos + 1) / every) + 1)
    bool value_norm;
    const float *slope, *bias;      // per head
    void* q;                  // [token][heads][q_pad], storage type: what logistic_prepare_kernel makes of the queries, zero beyond dim
    int q_pad;
    void *k, *v;              // cache: [slot][capacity][kv_heads][dim_pad], [..][vdim_pad]
    int capacity;
    void* out;                // [token][out_pitch], storage type (many tokens) ...
    int out_pitch;
    float* y;                 // ... or [token][heads * vdim], 32-bit (a step)
    int splits;               // step: shares of the keys
    float* part;              // step, splits > 1: [token][heads][splits][vdim]
    unsigned int* done;       // step, splits > 1: [token][head groups], zero between launches
};

// Norms of one token's queries, keys and values; the queries' temperature; keys and values go to the cache. One block per token; blocks beyond
// the last token clear the rows of the cache that follow it, so that kernels may multiply whole tiles of it by weights of zero.
template <typename T>
__global__ void __launch_bounds__(256) logistic_prepare_kernel(const __grid_constant__ LogisticArgs a) {
    __shared__ float red[8];
    const int z = blockIdx.x;
    const uint32_t slot = a.seq.pos_stride != 0 ? seq_of(a.seq, z) : 0, pos = seq_position(a.seq, a.pos, z);
    if (z >= a.tokens) {  // (of a prompt: its position is pos)
        if (pos >= static_cast<uint32_t>(a.capacity)) return;
        const size_t row = size_t(slot) * a.capacity + pos;
        for (int i = threadIdx.x; i < a.kv_heads * a.dim_pad; i += blockDim.x) static_cast<T*>(a.k)[row * a.kv_heads * a.dim_pad + i] = to_storage<T>(0.0f);
        for (int i = threadIdx.x; i < a.kv_heads * a.vdim_pad; i += blockDim.x) static_cast<T*>(a.v)[row * a.kv_heads * a.vdim_pad + i] = to_storage<T>(0.0f);
        return;
    }
    const float *q = a.p + size_t(z) * a.ld, *k = q + a.heads * a.dim, *v = k + a.kv_heads * a.dim;
    const int tid = threadIdx.x, nt = blockDim.x, nq = a.heads * a.dim, nk = a.kv_heads * a.dim;
    float iq = 1.0f, ik = 1.0f;
    if (a.q_norm != nullptr) {
        float s = 0.0f;
#pragma unroll 4
        for (int i = tid; i < nq; i += nt) s += q[i] * q[i];
        iq = 1.0f / sqrtf(block_sum(s, red) / static_cast<float>(nq) + a.eps);
    }
    if (a.k_norm != nullptr) {
        float s = 0.0f;
#pragma unroll 4
        for (int i = tid; i < nk; i += nt) s += k[i] * k[i];
        ik = 1.0f / sqrtf(block_sum(s, red) / static_cast<float>(nk) + a.eps);
    }
    const float temp = a.temp_coef != 0.0f ? 1.0f + a.temp_coef * logf(floorf(static_cast<float>(pos + 1) / a.temp_every) + 1.0f) : 1.0f;
    T* qo = static_cast<T*>(a.q) + size_t(z) * a.heads * a.q_pad;
#pragma unroll 4
    for (int i = tid; i < a.heads * a.q_pad; i += nt) {
        const int h = i / a.q_pad, e = i % a.q_pad, at = h * a.dim + e;
        qo[i] = to_storage<T>(e < a.dim ? __ldg(q + at) * iq * (a.q_norm != nullptr ? __ldg(a.q_norm + at) : 1.0f) * temp : 0.0f);
    }
    const size_t row = size_t(slot) * a.capacity + pos;
    T* ko = static_cast<T*>(a.k) + row * a.kv_heads * a.dim_pad;
    for (int i = tid; i < a.kv_heads * a.dim_pad; i += nt) {
        const int h = i / a.dim_pad, e = i % a.dim_pad, at = h * a.dim + e;
        ko[i] = to_storage<T>(e < a.dim ? __ldg(k + at) * ik * (a.k_norm != nullptr ? __ldg(a.k_norm + at) : 1.0f) : 0.0f);
    }
    T* vo = static_cast<T*>(a.v) + row * a.kv_heads * a.vdim_pad;
    const int warps = nt >> 5, lane = tid & 31;
    for (int h = tid >> 5; h < a.kv_heads; h += warps) {
        float s = 0.0f;
        for (int e = lane; e < a.vdim; e += 32) s += v[h * a.vdim + e] * v[h * a.vdim + e];
        const float iv = a.value_norm ? 1.0f / sqrtf(warp_sum(s) / static_cast<float>(a.vdim) + a.eps) : 1.0f;
        for (int e = lane; e < a.vdim_pad; e += 32) vo[h * a.vdim_pad + e] = to_storage<T>(e < a.vdim ? v[h * a.vdim + e] * iv : 0.0f);
    }
}

// ---- one query position per block ----------------------------------------------------------------------------------------------------------
// Up to H query heads of one kv head over a share of the keys; the last block of a position and head group to finish adds the shares up.
// 128 keys at a time: a few lanes per key make the weights, then a few lanes per key group add the values up. A decode step (OWN) makes the norms
// itself, takes its own key and value from the projections and appends them to the cache; the first cached keys and values are on their way
// before it waits for the projections. grid: (kv heads * head groups, splits, tokens or sequences)
constexpr int kLaThreads = 256, kLaKeys = 128;

inline int logistic_heads(int gqa) { return gqa <= 1 ? 1 : gqa <= 4 ? 4 : 8; }  // H the kernel is compiled for

inline int logistic_lanes(int pieces) { return pieces <= 1 ? 1 : pieces <= 2 ? 2 : pieces <= 4 ? 4 : pieces <= 8 ? 8 : pieces <= 16 ? 16 : pieces <= 32 ? 32 : 64; }
inline size_t logistic_step_smem(int heads, int dim_pad, int vdim, int vdim_pad, int elem) {
    const int lanes = logistic_lanes(vdim_pad * elem / 16), groups = lanes < 32 ? kLaThreads / 32 : kLaThreads / lanes;
    return (size_t(heads) * (dim_pad + kLaKeys + groups * vdim) + dim_pad + vdim_pad + kLaThreads) * 4;
}

template <typename T> struct Piece;  // 16 bytes of the storage type as floats
template <> struct Piece<bf16> {
    static constexpr int kN = 8;
    static __device__ __forceinline__ void get(const uint4& w, float (&f)[8]) {
        f[0] = __uint_as_float(w.x << 16), f[1] = __uint_as_float(w.x & 0xffff0000u), f[2] = __uint_as_float(w.y << 16), f[3] = __uint_as_float(w.y & 0xffff0000u);
        f[4] = __uint_as_float(w.z << 16), f[5] = __uint_as_float(w.z & 0xffff0000u), f[6] = __uint_as_float(w.w << 16), f[7] = __uint_as_float(w.w & 0xffff0000u);
    }
};
template <> struct Piece<float> {
    static constexpr int kN = 4;
    static __device__ __forceinline__ void get(const uint4& w, float (&f)[4]) { f[0] = __uint_as_float(w.x), f[1] = __uint_as_float(w.y), f[2] = __uint_as_float(w.z), f[3] = __uint_as_float(w.w); }
};

template <typename T, bool OWN, int H>
__global__ void __launch_bounds__(kLaThreads, H > 4 ? 1 : 2) logistic_step_kernel(const __grid_constant__ LogisticArgs a, int key_lanes, int value_lanes) {
    extern __shared__ __align__(16) float la_sm[];
    __shared__ bool last_block;
    __shared__ float sums[2][kLaThreads / 32], own_weight[H];
    constexpr int P = Piece<T>::kN;
    pdl_trigger();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int gqa = a.heads / a.kv_heads, groups = (gqa + H - 1) / H;
    const int kvh = blockIdx.x / groups, h0 = kvh * gqa + (blockIdx.x % groups) * H, nh = min(H, (kvh + 1) * gqa - h0);
    const int z = blockIdx.z, split = blockIdx.y;
    const uint32_t slot = a.seq.pos_stride != 0 ? seq_of(a.seq, z) : 0;
    const int pos = static_cast<int>(seq_position(a.seq, a.pos, z)), total = OWN ? pos : pos + 1;  // keys to be read from the cache
    const int per = (total + a.splits - 1) / a.splits, begin = min(split * per, total), end = min(begin + per, total);
    float *qs = la_sm, *ws = qs + H * a.dim_pad, *own_k = ws + H * kLaKeys, *own_v = own_k + a.dim_pad, *red = own_v + a.vdim_pad;
    const size_t krow = size_t(a.kv_heads) * a.dim_pad, vrow = size_t(a.kv_heads) * a.vdim_pad;
    T* ks = static_cast<T*>(a.k) + size_t(slot) * a.capacity * krow + kvh * a.dim_pad;
    T* vs = static_cast<T*>(a.v) + size_t(slot) * a.capacity * vrow + kvh * a.vdim_pad;
    const int kpieces = a.dim_pad / P, vpieces = a.vdim_pad / P;
    const int kl = lane & (key_lanes - 1), kg = (tid / key_lanes), kgroups = kLaThreads / key_lanes;        // key_lanes <= 32
    const int vl = tid & (value_lanes - 1), vg = tid / value_lanes, vgroups = kLaThreads / value_lanes;     // value_lanes <= 64
    uint4 kr[4], vr[8];
    auto fetch_keys = [&](int t0, int nt, int r0, int p) {
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int r = r0 + u * kgroups;
            kr[u] = r < nt && p < kpieces ? *reinterpret_cast<const uint4*>(ks + size_t(t0 + r) * krow + p * P) : make_uint4(0, 0, 0, 0);
        }
    };
    auto fetch_values = [&](int t0, int nt, int r0) {  // eight rows of this key group
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            const int r = r0 + u * vgroups;
            vr[u] = r < nt && vl < vpieces ? *reinterpret_cast<const uint4*>(vs + size_t(t0 + r) * vrow + vl * P) : make_uint4(0, 0, 0, 0);
        }
    };
    if (OWN) fetch_keys(begin, min(kLaKeys, end - begin), kg, kl), fetch_values(begin, min(kLaKeys, end - begin), vg);  // (written by earlier steps)
    pdl_wait();
    if (OWN) {
        const float *q = a.p + size_t(z) * a.ld, *k = q + a.heads * a.dim, *v = k + a.kv_heads * a.dim + kvh * a.vdim;
        const int nq = a.heads * a.dim, nk = a.kv_heads * a.dim;
        float sq = 0.0f, sk = 0.0f;
        if (a.q_norm != nullptr) {
#pragma unroll 8
            for (int i = tid; i < nq; i += kLaThreads) sq += q[i] * q[i];
        }
        if (a.k_norm != nullptr) {
#pragma unroll 4
            for (int i = tid; i < nk; i += kLaThreads) sk += k[i] * k[i];
        }
        sq = warp_sum(sq), sk = warp_sum(sk);
        if (lane == 0) sums[0][warp] = sq, sums[1][warp] = sk;
        __syncthreads();
        sq = sk = 0.0f;
#pragma unroll
        for (int w = 0; w < kLaThreads / 32; ++w) sq += sums[0][w], sk += sums[1][w];
        const float iq = a.q_norm != nullptr ? 1.0f / sqrtf(sq / static_cast<float>(nq) + a.eps) : 1.0f, ik = a.k_norm != nullptr ? 1.0f / sqrtf(sk / static_cast<float>(nk) + a.eps) : 1.0f;
        const float temp = a.temp_coef != 0.0f ? 1.0f + a.temp_coef * logf(floorf(static_cast<float>(pos + 1) / a.temp_every) + 1.0f) : 1.0f;
        for (int i = tid; i < nh * a.dim_pad; i += kLaThreads) {
            const int e = i % a.dim_pad, at = (h0 + i / a.dim_pad) * a.dim + e;
            qs[i] = e < a.dim ? round_to<T>(q[at] * iq * (a.q_norm != nullptr ? a.q_norm[at] : 1.0f) * temp) : 0.0f;
        }
        if (split == 0) {
            for (int e = tid; e < a.dim_pad; e += kLaThreads) own_k[e] = e < a.dim ? round_to<T>(k[kvh * a.dim + e] * ik * (a.k_norm != nullptr ? a.k_norm[kvh * a.dim + e] : 1.0f)) : 0.0f;
            if (warp == 7) {
                float sv = 0.0f;
                for (int e = lane; e < a.vdim; e += 32) sv += v[e] * v[e];
                const float iv = a.value_norm ? 1.0f / sqrtf(warp_sum(sv) / static_cast<float>(a.vdim) + a.eps) : 1.0f;
                for (int e = lane; e < a.vdim_pad; e += 32) own_v[e] = e < a.vdim ? round_to<T>(v[e] * iv) : 0.0f;
            }
            __syncthreads();
            if (warp < nh) {
                float s = 0.0f;
                for (int e = lane; e < a.dim_pad; e += 32) s = fmaf(qs[warp * a.dim_pad + e], own_k[e], s);
                s = warp_sum(s);
                if (lane == 0) own_weight[warp] = sigmoid_f(s * a.scale + a.bias[h0 + warp]);
            }
            if (blockIdx.x % groups == 0) {  // (no block of this launch reads this row of the cache)
                for (int e = tid; e < a.dim_pad; e += kLaThreads) ks[size_t(pos) * krow + e] = to_storage<T>(own_k[e]);
                for (int e = tid; e < a.vdim_pad; e += kLaThreads) vs[size_t(pos) * vrow + e] = to_storage<T>(own_v[e]);
            }
        }
    } else {
        for (int i = tid; i < nh * a.dim_pad; i += kLaThreads) qs[i] = from_storage(static_cast<const T*>(a.q)[(size_t(z) * a.heads + h0 + i / a.dim_pad) * a.q_pad + i % a.dim_pad]);
    }
    float acc[H][P];
#pragma unroll
    for (int h = 0; h < H; ++h)
#pragma unroll
        for (int e = 0; e < P; ++e) acc[h][e] = 0.0f;
    for (int t0 = begin; t0 < end; t0 += kLaKeys) {
        const int nt = min(kLaKeys, end - t0);
        const bool fetched = OWN && t0 == begin;
        if (!fetched) fetch_values(t0, nt, vg);
        __syncthreads();  // queries are there; weights of the tile before have been used
        for (int r0 = kg; r0 - kg < nt; r0 += 4 * kgroups) {
            float s[4][H];
#pragma unroll
            for (int u = 0; u < 4; ++u)
#pragma unroll
                for (int h = 0; h < H; ++h) s[u][h] = 0.0f;
            for (int p = kl; p < kpieces; p += key_lanes) {
                if (!(fetched && r0 == kg && p == kl)) fetch_keys(t0, nt, r0, p);
                float kf[4][P];
#pragma unroll
                for (int u = 0; u < 4; ++u) Piece<T>::get(kr[u], kf[u]);
#pragma unroll
                for (int h = 0; h < H; ++h)
                    if (h < nh) {
                        float q[P];
#pragma unroll
                        for (int e = 0; e < P; e += 4) *reinterpret_cast<float4*>(q + e) = *reinterpret_cast<const float4*>(qs + h * a.dim_pad + p * P + e);
#pragma unroll
                        for (int e = 0; e < P; ++e)
#pragma unroll
                            for (int u = 0; u < 4; ++u) s[u][h] = fmaf(q[e], kf[u][e], s[u][h]);
                    }
            }
            for (int o = key_lanes >> 1; o > 0; o >>= 1)
#pragma unroll
                for (int h = 0; h < H; ++h)
#pragma unroll
                    for (int u = 0; u < 4; ++u) s[u][h] += __shfl_xor_sync(0xffffffffu, s[u][h], o);
            if (kl == 0) {
#pragma unroll
                for (int h = 0; h < H; ++h)
#pragma unroll
                    for (int u = 0; u < 4; ++u) {
                        const int r = r0 + u * kgroups;
                        if (h < nh && r < nt) ws[h * kLaKeys + r] = s[u][h];
                    }
            }
        }
        __syncthreads();
        for (int i = tid; i < nh * kLaKeys; i += kLaThreads) {  // (entries beyond nt are not used)
            const int h = i / kLaKeys, r = i % kLaKeys;
            if (r < nt) ws[i] = sigmoid_f(ws[i] * a.scale - a.slope[h0 + h] * static_cast<float>(pos - t0 - r) + a.bias[h0 + h]);
        }
        __syncthreads();
        for (int r0 = vg; r0 < nt; r0 += 8 * vgroups) {
            if (r0 != vg) fetch_values(t0, nt, r0);
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                const int r = r0 + u * vgroups;
                if (r >= nt) break;
                float vf[P];
                Piece<T>::get(vr[u], vf);
#pragma unroll
                for (int h = 0; h < H; ++h)
                    if (h < nh) {
                        const float w = ws[h * kLaKeys + r];
#pragma unroll
                        for (int e = 0; e < P; ++e) acc[h][e] = fmaf(w, vf[e], acc[h][e]);
                    }
            }
        }
    }
    // sums of the key groups: those of a warp by shuffles, then through shared memory
    const int rows = value_lanes < 32 ? kLaThreads / 32 : vgroups, mine = value_lanes < 32 ? warp : vg;
    for (int o = 16; o >= value_lanes; o >>= 1)
#pragma unroll
        for (int h = 0; h < H; ++h)
#pragma unroll
            for (int e = 0; e < P; ++e) acc[h][e] += __shfl_xor_sync(0xffffffffu, acc[h][e], o);
    if (value_lanes >= 32 || lane < value_lanes) {
#pragma unroll
        for (int h = 0; h < H; ++h)
#pragma unroll
            for (int e = 0; e < P; ++e)
                if (h < nh && vl * P + e < a.vdim) red[(mine * H + h) * a.vdim + vl * P + e] = acc[h][e];
    }
    __syncthreads();
    for (int i = tid; i < nh * a.vdim; i += kLaThreads) {
        const int h = i / a.vdim, c = i % a.vdim;
        float s = OWN && split == 0 ? own_weight[h] * own_v[c] : 0.0f;
        for (int k = 0; k < rows; ++k) s += red[(k * H + h) * a.vdim + c];
        if (a.splits == 1) a.y[(size_t(z) * a.heads + h0 + h) * a.vdim + c] = s;
        else a.part[((size_t(z) * a.heads + h0 + h) * a.splits + split) * a.vdim + c] = s;
    }
    if (a.splits == 1) return;
    __threadfence();
    __syncthreads();
    unsigned int* counter = a.done + size_t(z) * gridDim.x + blockIdx.x;
    if (tid == 0) last_block = atomicAdd(counter, 1u) == static_cast<unsigned int>(a.splits) - 1;
    __syncthreads();
    if (!last_block) return;
    if (tid == 0) *counter = 0;
    __threadfence();
    // the shares that had keys; as many threads per four results as there are for them
    const int live = per > 0 ? max(1, (total + per - 1) / per) : 1, results = nh * a.vdim;
    const float* part0 = a.part + (size_t(z) * a.heads + h0) * a.splits * a.vdim;
    float* y0 = a.y + (size_t(z) * a.heads + h0) * a.vdim;
    if (a.vdim % 4 != 0) {
        for (int i = tid; i < results; i += kLaThreads) {
            const float* part = part0 + size_t(i / a.vdim) * a.splits * a.vdim + i % a.vdim;
            float s = 0.0f;
#pragma unroll 16
            for (int k = 0; k < live; ++k) s += __ldcg(part + size_t(k) * a.vdim);
            y0[i] = s;
        }
        return;
    }
    const int quads = results / 4, per_head = a.vdim / 4, teams = max(1, min(kLaThreads / quads, 8)), team = tid / quads;
    float4* team_sum = reinterpret_cast<float4*>(la_sm);  // [teams][quads]: at most kLaThreads
    if (teams == 1 || team < teams)
        for (int i = teams == 1 ? tid : tid % quads; i < quads; i += teams == 1 ? kLaThreads : quads) {
            const float4* part = reinterpret_cast<const float4*>(part0 + size_t(i / per_head) * a.splits * a.vdim) + i % per_head;
            float4 s = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll 8
            for (int k = teams == 1 ? 0 : team; k < live; k += teams) {
                const float4 f = __ldcg(part + size_t(k) * per_head);
                s.x += f.x, s.y += f.y, s.z += f.z, s.w += f.w;
            }
            if (teams == 1) reinterpret_cast<float4*>(y0)[i] = s;
            else team_sum[tid] = s;
        }
    if (teams == 1) return;
    __syncthreads();
    if (team != 0) return;
    float4 s = team_sum[tid];
    for (int t = 1; t < teams; ++t) {
        const float4 f = team_sum[t * quads + tid];
        s.x += f.x, s.y += f.y, s.z += f.z, s.w += f.w;
    }
    reinterpret_cast<float4*>(y0)[tid] = s;
}

// ---- many query positions on the tensor cores of a warp --------------------------------------------------------------------------------------
// For heads of more than 128 dimensions (logistic_attention_tc.cuh takes the others). 64 query positions of one head per block, keys in tiles of 64, fetched two tiles deep. A weight depends on its own score alone, so nothing is
// rescaled. Weights enter the second product as two bf16 terms. grid: (query tiles, heads)
constexpr int kLogisticMmaDims = 256;
template <int D>
__global__ void __launch_bounds__(kPmThreads) logistic_mma_kernel(const __grid_constant__ LogisticArgs a) {
    extern __shared__ __align__(16) unsigned char pm_sm[];
    constexpr int kPitch = D + 8;
    bf16* qs = reinterpret_cast<bf16*>(pm_sm);  // [64][kPitch]
    bf16* kv = qs + kPmRows * kPitch;           // two stages of keys and values, [64][kPitch] each
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, c = lane & 3;
    const int head = blockIdx.y, kvh = head / (a.heads / a.kv_heads), q0 = (gridDim.x - 1 - blockIdx.x) * kPmRows;
    const int pos0 = static_cast<int>(seq_position(a.seq, a.pos, 0));
    const int first = pos0 + q0, last = pos0 + min(q0 + kPmRows, a.tokens) - 1;
    const int dp = a.dim_pad, vp = a.vdim_pad;
    const bf16 *key0 = static_cast<const bf16*>(a.k) + size_t(kvh) * dp, *value0 = static_cast<const bf16*>(a.v) + size_t(kvh) * vp;
    const bf16* query0 = static_cast<const bf16*>(a.q) + size_t(head) * a.q_pad;
    for (int i = tid; i < kPmRows * (D / 8); i += kPmThreads) {
        const int r = i / (D / 8), p = i % (D / 8);
        const bool valid = q0 + r < a.tokens && p * 8 < dp;
        cp_async16(qs + r * kPitch + p * 8, query0 + (valid ? size_t(q0 + r) * a.heads * a.q_pad + p * 8 : 0), valid);
    }
    const int tiles = last / kPmKeys + 1;
    auto fetch = [&](int tile, int stage) {
        bf16 *ks = kv + stage * 2 * kPmKeys * kPitch, *vs = ks + kPmKeys * kPitch;
        for (int i = tid; i < kPmKeys * (D / 8); i += kPmThreads) {
            const int r = i / (D / 8), p = i % (D / 8), key = tile * kPmKeys + r;
            const size_t row = size_t(key <= last ? key : 0) * a.kv_heads;
            cp_async16(ks + r * kPitch + p * 8, key0 + row * dp + (p * 8 < dp ? p * 8 : 0), key <= last && p * 8 < dp);
            cp_async16(vs + r * kPitch + p * 8, value0 + row * vp + (p * 8 < vp ? p * 8 : 0), key <= last && p * 8 < vp);
        }
        cp_async_commit_group();
    };
    fetch(0, 0);
    float o[D / 8][4];
#pragma unroll
    for (int j = 0; j < D / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[j][e] = 0.0f;
    // exp(-score) = exp2(-log2(e) score): the sign and log2(e) go into the factors
    constexpr float kLog2e = 1.4426950408889634f;
    const float scale = -kLog2e * a.scale, slope = kLog2e * a.slope[head], bias = -kLog2e * a.bias[head];
    const int row0 = first + warp * 16 + g;
    for (int tile = 0; tile < tiles; ++tile) {
        if (tile + 1 < tiles) {
            fetch(tile + 1, (tile + 1) & 1);
            cp_async_wait_group<1>();
        } else {
            cp_async_wait_group<0>();
        }
        __syncthreads();
        const bf16 *ks = kv + (tile & 1) * 2 * kPmKeys * kPitch, *vs = ks + kPmKeys * kPitch;
        float s[kPmKeys / 8][4];
#pragma unroll
        for (int j = 0; j < kPmKeys / 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) s[j][e] = 0.0f;
#pragma unroll
        for (int k = 0; k < D / 16; ++k) {
            uint32_t q[4];  // (too many to stay in registers)
            load_frag_a(q, qs + warp * 16 * kPitch + k * 16, kPitch);
#pragma unroll
            for (int j = 0; j < kPmKeys / 8; j += 2) {
                uint32_t b[4];
                load_frag_bt(b, ks + j * 8 * kPitch + k * 16, kPitch);
                mma_16816(s[j], q, b[0], b[1]);
                mma_16816(s[j + 1], q, b[2], b[3]);
            }
        }
        const int k0 = tile * kPmKeys;
        const bool open = k0 + kPmKeys - 1 <= first;  // every row sees the whole tile
#pragma unroll
        for (int j = 0; j < kPmKeys / 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int back = row0 + (e >> 1) * 8 - (k0 + j * 8 + 2 * c + (e & 1));
                const float w = __fdividef(1.0f, 1.0f + fast_exp2(fmaf(slope, static_cast<float>(back), fmaf(s[j][e], scale, bias))));
                s[j][e] = open || back >= 0 ? w : 0.0f;
            }
#pragma unroll
        for (int k = 0; k < kPmKeys / 16; ++k) {  // the weights of 16 keys are an A operand as they lie
            uint32_t ph[4], pl[4];
            split_bf16(s[2 * k][0], s[2 * k][1], &ph[0], &pl[0]), split_bf16(s[2 * k][2], s[2 * k][3], &ph[1], &pl[1]);
            split_bf16(s[2 * k + 1][0], s[2 * k + 1][1], &ph[2], &pl[2]), split_bf16(s[2 * k + 1][2], s[2 * k + 1][3], &ph[3], &pl[3]);
#pragma unroll
            for (int j = 0; j < D / 8; j += 2) {
                uint32_t b[4];
                load_frag_b(b, vs + k * 16 * kPitch + j * 8, kPitch);
                mma_16816(o[j], ph, b[0], b[1]), mma_16816(o[j + 1], ph, b[2], b[3]);
                mma_16816(o[j], pl, b[0], b[1]), mma_16816(o[j + 1], pl, b[2], b[3]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        const int t = q0 + warp * 16 + g + 8 * h;
        if (t >= a.tokens) continue;
        bf16* out = static_cast<bf16*>(a.out) + size_t(t) * a.out_pitch + size_t(head) * a.vdim;
#pragma unroll
        for (int j = 0; j < D / 8; ++j)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int v = j * 8 + 2 * c + e;
                if (v < a.vdim) out[v] = __float2bfloat16_rn(o[j][2 * h + e]);
            }
    }
}

}  // namespace qtb
