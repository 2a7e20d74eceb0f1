// The attention of pooled_attention.cuh for many query tokens, on the tensor cores of a warp: 64 query positions of one head per block, keys in
// tiles of 64 - first the pooled blocks, then the tokens of the windows - fetched two tiles deep. Scores, running maxima and weights are 32-bit;
// the weights enter the second product as two bf16 terms.
#pragma once
#include "mma_bf16.cuh"
#include "pooled_attention.cuh"

namespace qtb {

constexpr int kPmRows = 64, kPmKeys = 64, kPmThreads = 128;

// Padded head size the kernel is compiled for, 0 if the heads are too large for it.
inline int pooled_mma_dims(int dim, int vdim) {
    const int d = dim > vdim ? dim : vdim;
    return d <= 32 ? 32 : d <= 64 ? 64 : d <= 128 ? 128 : 0;
}
inline size_t pooled_mma_smem(int dims) { return size_t(kPmRows + 4 * kPmKeys) * (dims + 8) * 2; }

__device__ __forceinline__ float fast_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// grid: (query tiles, heads). The launch's keys and values are in the cache (pooled_append_kernel).
template <int D>
__global__ void __launch_bounds__(kPmThreads) pooled_attention_mma_kernel(const __grid_constant__ PooledAttnArgs a) {
    extern __shared__ __align__(16) unsigned char pm_sm[];
    constexpr int kPitch = D + 8;
    bf16* qs = reinterpret_cast<bf16*>(pm_sm);  // [64][kPitch]
    bf16* kv = qs + kPmRows * kPitch;           // two stages of keys and values, [64][kPitch] each
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, c = lane & 3;
    const int head = blockIdx.y, kvh = head / (a.heads / a.kv_heads), q0 = (gridDim.x - 1 - blockIdx.x) * kPmRows;
    const int pos0 = static_cast<int>(seq_position(a.seq, a.pos, 0));
    const int first = pos0 + q0, last = pos0 + min(q0 + kPmRows, a.tokens) - 1;
    const int dp = a.dim_pad, vp = a.vdim_pad;
    const bf16* ring_k = static_cast<const bf16*>(a.cache.k) + size_t(kvh) * dp;
    const bf16* ring_v = static_cast<const bf16*>(a.cache.v) + size_t(kvh) * vp;
    const bf16* pool_k = static_cast<const bf16*>(a.cache.pk) + size_t(kvh) * dp;
    const bf16* pool_v = static_cast<const bf16*>(a.cache.pv) + size_t(kvh) * vp;
    for (int i = tid; i < kPmRows * D; i += kPmThreads) {
        const int r = i / D, e = i % D;
        qs[r * kPitch + e] = __float2bfloat16_rn(e < a.dim && q0 + r < a.tokens ? a.p[size_t(q0 + r) * a.ld + head * a.dim + e] : 0.0f);
    }
    const int nb = pooled_blocks_seen(last, a.window, a.pool), lo = max(0, first - a.window + 1);  // blocks and tokens that any row sees
    const int pool_tiles = (nb + kPmKeys - 1) / kPmKeys, tiles = pool_tiles + (last - lo + kPmKeys) / kPmKeys;
    auto fetch = [&](int tile, int stage) {
        bf16 *ks = kv + stage * 2 * kPmKeys * kPitch, *vs = ks + kPmKeys * kPitch;
        const bool pooled = tile < pool_tiles;
        const int k0 = pooled ? tile * kPmKeys : lo + (tile - pool_tiles) * kPmKeys;
        for (int i = tid; i < kPmKeys * (D / 8); i += kPmThreads) {
            const int r = i / (D / 8), p = i % (D / 8), key = k0 + r;
            const bool valid = pooled ? key < nb : key <= last;
            const size_t row = size_t(valid ? (pooled ? key : key % a.cache.ring) : 0) * a.kv_heads;
            cp_async16(ks + r * kPitch + p * 8, (pooled ? pool_k : ring_k) + row * dp + (p * 8 < dp ? p * 8 : 0), valid && p * 8 < dp);
            cp_async16(vs + r * kPitch + p * 8, (pooled ? pool_v : ring_v) + row * vp + (p * 8 < vp ? p * 8 : 0), valid && p * 8 < vp);
        }
        cp_async_commit_group();
    };
    fetch(0, 0);
    __syncthreads();
    uint32_t q[D / 16][4];
#pragma unroll
    for (int ks = 0; ks < D / 16; ++ks) load_frag_a(q[ks], qs + warp * 16 * kPitch + ks * 16, kPitch);
    float o[D / 8][4];
#pragma unroll
    for (int j = 0; j < D / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[j][e] = 0.0f;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
    int row_pos[2], row_nb[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) row_pos[h] = first + warp * 16 + g + 8 * h, row_nb[h] = pooled_blocks_seen(row_pos[h], a.window, a.pool);
    const int first_nb = pooled_blocks_seen(first, a.window, a.pool);
    const float to_exp2 = a.scale * 1.4426950408889634f;  // log2(e)
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
        for (int k = 0; k < D / 16; ++k)
#pragma unroll
            for (int j = 0; j < kPmKeys / 8; j += 2) {
                uint32_t b[4];
                load_frag_bt(b, ks + j * 8 * kPitch + k * 16, kPitch);
                mma_16816(s[j], q[k], b[0], b[1]);
                mma_16816(s[j + 1], q[k], b[2], b[3]);
            }
        const bool pooled = tile < pool_tiles;
        const int k0 = pooled ? tile * kPmKeys : lo + (tile - pool_tiles) * kPmKeys;
        float mx[2] = {m[0], m[1]};
        const bool open = pooled ? k0 + kPmKeys <= first_nb : k0 + kPmKeys - 1 <= first && k0 > first + kPmRows - 1 - a.window;  // every row sees the whole tile
        if (open) {
#pragma unroll
            for (int j = 0; j < kPmKeys / 8; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) s[j][e] *= to_exp2, mx[e >> 1] = fmaxf(mx[e >> 1], s[j][e]);
        } else {
#pragma unroll
            for (int j = 0; j < kPmKeys / 8; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int h = e >> 1, key = k0 + j * 8 + 2 * c + (e & 1);
                    const bool seen = pooled ? key < row_nb[h] : key <= row_pos[h] && key > row_pos[h] - a.window;
                    s[j][e] = seen ? s[j][e] * to_exp2 : -INFINITY;
                    mx[h] = fmaxf(mx[h], s[j][e]);
                }
        }
        float fac[2], m_safe[2];
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
            mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
            fac[h] = mx[h] == -INFINITY ? 1.0f : exp2f(m[h] - mx[h]);  // nothing seen so far: nothing to rescale
            m[h] = mx[h];
            m_safe[h] = mx[h] == -INFINITY ? 0.0f : mx[h];
            l[h] *= fac[h];
        }
#pragma unroll
        for (int j = 0; j < D / 8; ++j) o[j][0] *= fac[0], o[j][1] *= fac[0], o[j][2] *= fac[1], o[j][3] *= fac[1];
#pragma unroll
        for (int j = 0; j < kPmKeys / 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int h = e >> 1;
                s[j][e] = fast_exp2(s[j][e] - m_safe[h]);  // 0 for a key that is not seen
                l[h] += s[j][e];
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
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 1);
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 2);
        const int t = q0 + warp * 16 + g + 8 * h;
        if (t >= a.tokens) continue;
        const float gate = a.head_gate ? sigmoid_f(a.p[size_t(t) * a.ld + a.heads * a.dim + a.kv_heads * (a.dim + a.vdim) + head]) : 1.0f, f = gate / l[h];
        float* y = a.y + size_t(t) * a.heads * a.vdim + size_t(head) * a.vdim;
#pragma unroll
        for (int j = 0; j < D / 8; ++j)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int v = j * 8 + 2 * c + e;
                if (v < a.vdim) y[v] = o[j][2 * h + e] * f;
            }
    }
}

}  // namespace qtb
