// Attention over a sliding window and pooled blocks. Position i sees the tokens j with 0 <= i - j < window and, beside them, one key and
// one value for each block of `pool` tokens that lies wholly before the window (block b: positions b pool .. (b + 1) pool - 1, seen when
// (b + 1) pool - 1 <= i - window): the means of the block's keys and values as the cache holds them. Tokens between the last visible block
// and the window are not seen. One softmax over blocks and tokens, 32-bit scores and weights.
//
// The cache of a layer and sequence: a ring of the last `ring` keys and values (position p in slot p % ring; ring >= window + the longest
// launch), and the pooled keys and values from the start of the sequence. Rows are [kv head][dim padded to 8], storage type. A block's mean is
// written by the launch that brings its last token.
#pragma once
#include "dense_gemv.cuh"

namespace qtb {

struct PooledCache {
    void *k, *v;              // [slot][ring][kv_heads][dim_pad], [..][vdim_pad]
    void *pk, *pv;            // [slot][blocks][kv_heads][..]
    int ring, blocks;         // blocks: capacity (0 without pooling)
};

struct PooledAttnArgs {
    int tokens;               // consecutive tokens of a sequence (1: a decode step, sequences in gridDim.z)
    const uint32_t* pos;
    SeqIndex seq;
    const float* p;           // projections [token][ld]: q | k | v | g
    int ld;
    int heads, kv_heads, dim, vdim, dim_pad, vdim_pad;
    int window, pool;         // pool 0: no pooled blocks
    float scale;
    bool head_gate;
    PooledCache cache;
    float* y;                 // [token][heads * vdim]
    // split form
    int splits;
    float *part_acc, *part_ml;      // [token][heads][splits][vdim], [token][heads][splits][2]
    unsigned int* done;             // [token][head groups], zero between launches
};

__device__ __forceinline__ int pooled_blocks_seen(int pos, int window, int pool) { return pool > 0 && pos - window + 1 > 0 ? (pos - window + 1) / pool : 0; }

// Writes keys and values of the launch's tokens to the ring and the means of the blocks that become complete.
// grid: (aligned groups of tokens, kv heads, sequences); the groups are `pool` tokens long (64 without pooling).
template <typename T>
__global__ void __launch_bounds__(256) pooled_append_kernel(const __grid_constant__ PooledAttnArgs a) {
    const int z = blockIdx.z, kvh = blockIdx.y, unit = a.pool > 0 ? a.pool : 64;
    const uint32_t slot = a.seq.pos_stride != 0 ? seq_of(a.seq, z) : 0;
    const int pos0 = static_cast<int>(seq_position(a.seq, a.pos, z)), end = pos0 + a.tokens;
    const int block = pos0 / unit + blockIdx.x, b0 = block * unit, b1 = b0 + unit;
    if (b0 >= end) return;
    const bool complete = a.pool > 0 && b1 <= end;
    const float* rows = a.p + size_t(z) * a.tokens * a.ld;
    for (int c = threadIdx.x; c < a.dim_pad + a.vdim_pad; c += blockDim.x) {
        const bool key = c < a.dim_pad;
        const int e = key ? c : c - a.dim_pad, width = key ? a.dim : a.vdim, pad = key ? a.dim_pad : a.vdim_pad;
        const int src = a.heads * a.dim + (key ? kvh * a.dim : a.kv_heads * a.dim + kvh * a.vdim) + e;
        T* ring = static_cast<T*>(key ? a.cache.k : a.cache.v) + (size_t(slot) * a.cache.ring * a.kv_heads + kvh) * pad + e;
        const size_t step = size_t(a.kv_heads) * pad;
        float sum = 0.0f;
        if (complete)
            for (int j = b0; j < min(pos0, b1); ++j) sum += from_storage(ring[size_t(j % a.cache.ring) * step]);
        for (int j0 = max(b0, pos0); j0 < min(b1, end); j0 += 8) {
            float v[8];  // eight loads in flight
#pragma unroll
            for (int k = 0; k < 8; ++k) v[k] = e < width && j0 + k < min(b1, end) ? rows[size_t(j0 + k - pos0) * a.ld + src] : 0.0f;
#pragma unroll
            for (int k = 0; k < 8; ++k)
                if (j0 + k < min(b1, end)) {
                    const T t = to_storage<T>(v[k]);
                    ring[size_t((j0 + k) % a.cache.ring) * step] = t;
                    sum += from_storage(t);
                }
        }
        if (complete) {
            T* pool = static_cast<T*>(key ? a.cache.pk : a.cache.pv) + ((size_t(slot) * a.cache.blocks + block) * a.kv_heads + kvh) * pad + e;
            *pool = to_storage<T>(sum / static_cast<float>(a.pool));
        }
    }
}

constexpr int kPaThreads = 256, kPaTile = 64, kPaHeads = 8;  // keys per tile; query heads per block

inline size_t pooled_attn_smem(int dim_pad, int vdim_pad, int elem) {
    return size_t(kPaHeads) * dim_pad * 4 + size_t(kPaTile) * (size_t(dim_pad) * elem + 16) + size_t(kPaTile) * vdim_pad * elem + size_t(kPaHeads) * kPaTile * 4 +
           size_t(kPaHeads) * 2 * kPaThreads * 4 + 64;
}

__device__ __forceinline__ float dot_key(const bf16* k, const float* q, int dim_pad) {
    float s = 0.0f;
    for (int c = 0; c < dim_pad; c += 8) {
        const uint4 w = *reinterpret_cast<const uint4*>(k + c);
        const float4 a = *reinterpret_cast<const float4*>(q + c), b = *reinterpret_cast<const float4*>(q + c + 4);
        s = fmaf(__uint_as_float(w.x << 16), a.x, s), s = fmaf(__uint_as_float(w.x & 0xffff0000u), a.y, s);
        s = fmaf(__uint_as_float(w.y << 16), a.z, s), s = fmaf(__uint_as_float(w.y & 0xffff0000u), a.w, s);
        s = fmaf(__uint_as_float(w.z << 16), b.x, s), s = fmaf(__uint_as_float(w.z & 0xffff0000u), b.y, s);
        s = fmaf(__uint_as_float(w.w << 16), b.z, s), s = fmaf(__uint_as_float(w.w & 0xffff0000u), b.w, s);
    }
    return s;
}
__device__ __forceinline__ float dot_key(const float* k, const float* q, int dim_pad) {
    float s = 0.0f;
    for (int c = 0; c < dim_pad; c += 4) {
        const float4 w = *reinterpret_cast<const float4*>(k + c), a = *reinterpret_cast<const float4*>(q + c);
        s = fmaf(w.x, a.x, s), s = fmaf(w.y, a.y, s), s = fmaf(w.z, a.z, s), s = fmaf(w.w, a.w, s);
    }
    return s;
}

__device__ __forceinline__ void attn_copy16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(dst))), "l"(src) : "memory");
}

// One query position per block: up to eight query heads of one kv head over a share (split) of the visible keys; the last block of a
// position and head group to finish adds the shares up. A decode step (APPEND) also stores its own key and value, and the mean of a block
// that this token completes. grid: (kv heads * head groups, splits, tokens or sequences)
template <typename T, bool APPEND>
__global__ void __launch_bounds__(kPaThreads) pooled_attention_kernel(const __grid_constant__ PooledAttnArgs a) {
    extern __shared__ __align__(16) float pa_sm[];
    pdl_trigger();
    __shared__ float m_run[kPaHeads], l_run[kPaHeads], fac[kPaHeads];
    __shared__ bool last_block;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int gqa = a.heads / a.kv_heads, groups = (gqa + kPaHeads - 1) / kPaHeads;
    const int kvh = blockIdx.x / groups, h0 = kvh * gqa + (blockIdx.x % groups) * kPaHeads, nh = min(kPaHeads, (kvh + 1) * gqa - h0);
    const int z = blockIdx.z, split = blockIdx.y;
    const uint32_t slot = a.seq.pos_stride != 0 ? seq_of(a.seq, z) : 0;
    const int pos = static_cast<int>(seq_position(a.seq, a.pos, z));
    const int dp = a.dim_pad, vp = a.vdim_pad;
    const int kpitch = dp * sizeof(T) + 16;  // bytes: a thread per key reads 16 bytes of its own row, conflict-free
    float* qs = pa_sm;                                                                   // [kPaHeads][dp]
    unsigned char* kt = reinterpret_cast<unsigned char*>(qs + kPaHeads * dp);            // [kPaTile][kpitch]
    T* vt = reinterpret_cast<T*>(kt + kPaTile * kpitch);                                 // [kPaTile][vp]
    float* sc = reinterpret_cast<float*>(vt + kPaTile * vp);                             // [kPaHeads][kPaTile]
    float* red = sc + kPaHeads * kPaTile;                                                // [key groups][kPaHeads][vstride]
    const float* prow = a.p + size_t(z) * a.ld;
    if (tid < kPaHeads) m_run[tid] = -INFINITY, l_run[tid] = 0.0f;
    const int nb = pooled_blocks_seen(pos, a.window, a.pool), lo = max(0, pos - a.window + 1), total = nb + pos - lo + 1;
    const int per = ((total + a.splits - 1) / a.splits + kPaTile - 1) / kPaTile * kPaTile;
    const int begin = min(split * per, total), end = min(begin + per, total);
    const T* ring_k = static_cast<const T*>(a.cache.k) + (size_t(slot) * a.cache.ring * a.kv_heads + kvh) * dp;
    const T* ring_v = static_cast<const T*>(a.cache.v) + (size_t(slot) * a.cache.ring * a.kv_heads + kvh) * vp;
    const T* pool_k = static_cast<const T*>(a.cache.pk) + (size_t(slot) * a.cache.blocks * a.kv_heads + kvh) * dp;
    const T* pool_v = static_cast<const T*>(a.cache.pv) + (size_t(slot) * a.cache.blocks * a.kv_heads + kvh) * vp;
    const int src_k = a.heads * a.dim + kvh * a.dim, src_v = a.heads * a.dim + a.kv_heads * a.dim + kvh * a.vdim;
    // value columns: thread (key group kg, column vc); columns beyond 128 take a second turn
    const int vcols = vp <= 32 ? 32 : vp <= 64 ? 64 : 128, kgroups = kPaThreads / vcols, kg = tid / vcols, vc = tid % vcols;
    const int vstride = vp > 128 ? 256 : vcols;
    float acc[kPaHeads][2] = {};
    constexpr int kPer = 16 / sizeof(T);
    const int kvec = dp / kPer, vvec = vp / kPer;
    auto fetch = [&](int t0) {  // keys and values of a tile; a decode step's own token is not in the cache yet
        const int nt = min(kPaTile, end - t0);
#pragma unroll 4
        for (int i = tid; i < nt * (kvec + vvec); i += kPaThreads) {
            const int r = i / (kvec + vvec), c = i % (kvec + vvec), key = t0 + r;
            const bool pooled = key < nb, is_k = c < kvec;
            const int token = lo + key - nb;
            if (APPEND && !pooled && token == pos) continue;
            const size_t row = size_t(pooled ? key : token % a.cache.ring) * a.kv_heads;
            const T* from = is_k ? (pooled ? pool_k : ring_k) + row * dp + c * kPer : (pooled ? pool_v : ring_v) + row * vp + (c - kvec) * kPer;
            attn_copy16(is_k ? static_cast<void*>(kt + r * kpitch + c * 16) : static_cast<void*>(vt + r * vp + (c - kvec) * kPer), from);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (begin < end) fetch(begin);  // (cached by earlier steps, or by the launch before where this is a prompt's)
    pdl_wait();
    for (int i = tid; i < kPaHeads * dp; i += kPaThreads) {
        const int h = i / dp, c = i % dp;
        qs[i] = h < nh && c < a.dim ? round_to<T>(prow[(h0 + h) * a.dim + c]) : 0.0f;
    }
    for (int t0 = begin; t0 < end; t0 += kPaTile) {
        const int nt = min(kPaTile, end - t0);
        if (t0 != begin) {
            __syncthreads();
            fetch(t0);
        }
        if (APPEND && pos - lo + nb >= t0 && pos - lo + nb < t0 + nt) {  // this step's own token: from the projections
            const int r = pos - lo + nb - t0;
            for (int e = tid; e < dp + vp; e += kPaThreads) {
                if (e < dp) reinterpret_cast<T*>(kt + r * kpitch)[e] = to_storage<T>(e < a.dim ? prow[src_k + e] : 0.0f);
                else vt[r * vp + e - dp] = to_storage<T>(e - dp < a.vdim ? prow[src_v + e - dp] : 0.0f);
            }
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        for (int i = tid; i < kPaTile * nh; i += kPaThreads) {
            const int r = i % kPaTile, h = i / kPaTile;
            sc[h * kPaTile + r] = r < nt ? dot_key(reinterpret_cast<const T*>(kt + r * kpitch), qs + h * dp, dp) * a.scale : -INFINITY;
        }
        __syncthreads();
        for (int h = warp; h < nh; h += kPaThreads / 32) {
            float s0 = sc[h * kPaTile + lane], s1 = sc[h * kPaTile + 32 + lane], mx = fmaxf(s0, s1);
            for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float m_old = m_run[h], m_new = fmaxf(m_old, mx);
            s0 = expf(s0 - m_new), s1 = expf(s1 - m_new);
            const float sum = warp_sum(s0 + s1);
            sc[h * kPaTile + lane] = s0, sc[h * kPaTile + 32 + lane] = s1;
            if (lane == 0) {
                const float f = expf(m_old - m_new);
                fac[h] = f, m_run[h] = m_new, l_run[h] = l_run[h] * f + sum;
            }
        }
        __syncthreads();
#pragma unroll
        for (int h = 0; h < kPaHeads; ++h)
            if (h < nh) acc[h][0] *= fac[h], acc[h][1] *= fac[h];
        for (int r = kg; r < nt; r += kgroups) {
            const float w0 = vc < vp ? from_storage(vt[r * vp + vc]) : 0.0f, w1 = vc + 128 < vp ? from_storage(vt[r * vp + vc + 128]) : 0.0f;
#pragma unroll
            for (int h = 0; h < kPaHeads; ++h)
                if (h < nh) {
                    const float p = sc[h * kPaTile + r];
                    acc[h][0] = fmaf(p, w0, acc[h][0]), acc[h][1] = fmaf(p, w1, acc[h][1]);
                }
        }
    }
    // the key groups' sums, head by head
    __syncthreads();
#pragma unroll
    for (int h = 0; h < kPaHeads; ++h)
        if (h < nh) {
            red[(kg * kPaHeads + h) * vstride + vc] = acc[h][0];
            if (vstride == 256) red[(kg * kPaHeads + h) * vstride + 128 + vc] = acc[h][1];
        }
    __syncthreads();
    for (int i = tid; i < nh * a.vdim; i += kPaThreads) {
        const int h = i / a.vdim, v = i % a.vdim, head = h0 + h;
        float s = 0.0f;
        for (int g = 0; g < kgroups; ++g) s += red[(g * kPaHeads + h) * vstride + v];
        if (a.splits == 1) {
            const float gate = a.head_gate ? sigmoid_f(prow[a.heads * a.dim + a.kv_heads * (a.dim + a.vdim) + head]) : 1.0f;
            a.y[size_t(z) * a.heads * a.vdim + size_t(head) * a.vdim + v] = s / l_run[h] * gate;
        } else {
            const size_t at = (size_t(z) * a.heads + head) * a.splits + split;
            a.part_acc[at * a.vdim + v] = s;
            if (v == 0) a.part_ml[at * 2] = m_run[h], a.part_ml[at * 2 + 1] = l_run[h];
        }
    }
    if (APPEND && split == 0 && blockIdx.x % groups == 0) {
        // this token's row of the ring, and the mean of the block it completes. No block of this launch reads either: the slot's previous
        // token has left the window, and a block is seen only once it lies before the window.
        const bool complete = a.pool > 0 && (pos + 1) % a.pool == 0;
        for (int c = tid; c < dp + vp; c += kPaThreads) {
            const bool key = c < dp;
            const int e = key ? c : c - dp, width = key ? a.dim : a.vdim, pad = key ? dp : vp;
            T* ring = const_cast<T*>(key ? ring_k : ring_v) + e;
            const size_t step = size_t(a.kv_heads) * pad;
            const T v = to_storage<T>(e < width ? prow[(key ? src_k : src_v) + e] : 0.0f);
            if (complete) {
                float sum = 0.0f;
                for (int j = pos + 1 - a.pool; j < pos; ++j) sum += from_storage(ring[size_t(j % a.cache.ring) * step]);
                T* pool = const_cast<T*>(key ? pool_k : pool_v) + size_t(pos / a.pool) * step + e;
                *pool = to_storage<T>((sum + from_storage(v)) / static_cast<float>(a.pool));
            }
            ring[size_t(pos % a.cache.ring) * step] = v;
        }
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
    // factors of the shares, then the sums
    float* part = sc;  // [nh][splits]; kPaHeads x kPaTile floats hold at most 64 shares a head
    for (int h = warp; h < nh; h += kPaThreads / 32) {
        const float* ml = a.part_ml + (size_t(z) * a.heads + h0 + h) * a.splits * 2;
        float mk[2], lk[2], m = -INFINITY;
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const int i = lane + 32 * k;
            mk[k] = i < a.splits ? __ldcg(ml + 2 * i) : -INFINITY, lk[k] = i < a.splits ? __ldcg(ml + 2 * i + 1) : 0.0f;
            m = fmaxf(m, mk[k]);
        }
        for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
        float l = 0.0f;
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            mk[k] = mk[k] == -INFINITY ? 0.0f : expf(mk[k] - m);  // an empty share counts nothing
            l = fmaf(lk[k], mk[k], l);
        }
        l = warp_sum(l);
        const float gate = a.head_gate ? sigmoid_f(prow[a.heads * a.dim + a.kv_heads * (a.dim + a.vdim) + h0 + h]) : 1.0f;
#pragma unroll
        for (int k = 0; k < 2; ++k)
            if (lane + 32 * k < a.splits) part[h * kPaTile + lane + 32 * k] = mk[k] * gate / l;
    }
    __syncthreads();
    const float* acc0 = a.part_acc + (size_t(z) * a.heads + h0) * a.splits * a.vdim;
    float* y0 = a.y + size_t(z) * a.heads * a.vdim + size_t(h0) * a.vdim;
    if (a.vdim % 4 == 0) {
        const int quads = a.vdim / 4;
        for (int i = tid; i < nh * quads; i += kPaThreads) {
            const int h = i / quads, v = i % quads * 4;
            float4 s = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll 12
            for (int k = 0; k < a.splits; ++k) {
                const float4 p = __ldcg(reinterpret_cast<const float4*>(acc0 + (size_t(h) * a.splits + k) * a.vdim + v));
                const float f = part[h * kPaTile + k];
                s.x = fmaf(p.x, f, s.x), s.y = fmaf(p.y, f, s.y), s.z = fmaf(p.z, f, s.z), s.w = fmaf(p.w, f, s.w);
            }
            *reinterpret_cast<float4*>(y0 + h * a.vdim + v) = s;
        }
        return;
    }
    for (int i = tid; i < nh * a.vdim; i += kPaThreads) {
        const int h = i / a.vdim, v = i % a.vdim;
        float s = 0.0f;
#pragma unroll 8
        for (int k = 0; k < a.splits; ++k) s = fmaf(__ldcg(acc0 + (size_t(h) * a.splits + k) * a.vdim + v), part[h * kPaTile + k], s);
        y0[h * a.vdim + v] = s;
    }
}

}  // namespace qtb
