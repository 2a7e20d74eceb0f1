// Retention (gated_scan.cuh) over many tokens. With one decay a per head the state after a chunk of T tokens is a^T S + U, where U depends on the
// chunk's own keys and values only, and
//
//   y_t = a^(t + 1) q_t S + sum over s <= t of a^(t - s) (q_t . k_s) v_s        t, s: places in the chunk
//
// so the chunks need not follow one another: U of every chunk at once, then S at every chunk's start (one multiply-add per element and chunk), then
// every chunk's outputs at once. 64 tokens a chunk, products on the warp tensor cores; queries, keys, states and decayed weights go in as two bf16
// terms, values as one. The last kernel also divides each head's output by its root mean square and multiplies it by silu(g).
#pragma once
#include "gated_scan.cuh"
#include "mma_bf16.cuh"

namespace qtb {

constexpr int kRetT = 64;      // tokens of a chunk
constexpr int kRetV = 64;      // value columns per block of the first kernel, and per turn of the last

// Compiled sizes: rows of the state and value columns, 0 if a head is too large.
inline int retention_rows(int dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : dim <= 128 ? 128 : dim <= 256 ? 256 : 0; }
inline int retention_cols(int vdim) { return vdim <= 64 ? 64 : vdim <= 128 ? 128 : vdim <= 256 ? 256 : 0; }
inline int retention_chunks(int tokens) { return (tokens + kRetT - 1) / kRetT; }

struct RetentionWork {
    float* u;              // [head][chunk][v_pad][rows]
    bf16 *s_hi, *s_lo;     // the state before each chunk, same order
    int rows, v_pad;
};
inline size_t retention_work(char* base, int heads, int dim, int vdim, int tokens, RetentionWork* w) {
    w->rows = retention_rows(dim), w->v_pad = retention_cols(vdim);
    const size_t n = size_t(heads) * retention_chunks(tokens) * w->v_pad * w->rows;
    w->u = reinterpret_cast<float*>(base), w->s_hi = reinterpret_cast<bf16*>(base + n * 4), w->s_lo = w->s_hi + n;
    return n * 8;
}

struct RetentionArgs {
    ScanArgs scan;
    RetentionWork work;
    float eps;             // of the heads' norm
    void* out;             // [token][out_pitch], bf16
    int out_pitch;
};

// powers a^0 .. a^T of a head's decay
__device__ __forceinline__ void decay_powers(float decay, float* pw) {
    for (int i = threadIdx.x; i <= kRetT; i += blockDim.x) pw[i] = i == 0 ? 1.0f : decay > 0.0f ? exp2f(static_cast<float>(i) * log2f(decay)) : 0.0f;
}
__device__ __forceinline__ void put_split(bf16* hi, bf16* lo, int at, float v) {
    const bf16 h = __float2bfloat16_rn(v);
    hi[at] = h, lo[at] = __float2bfloat16_rn(v - __bfloat162float(h));
}

// U of every chunk. grid: (heads, chunks, ceil(vdim / 64)), 128 threads; a warp owns 16 value columns
template <int N> __host__ __device__ constexpr size_t retention_state_smem() { return size_t(2 * kRetT) * (N + 8) * 2 + size_t(kRetT) * (kRetV + 8) * 2; }
template <int N>
__global__ void __launch_bounds__(128) retention_state_kernel(const __grid_constant__ RetentionArgs r) {
    extern __shared__ __align__(16) unsigned char rt_sm[];
    __shared__ float pw[kRetT + 1];
    const ScanArgs& a = r.scan;
    constexpr int kPitch = N + 8, kVPitch = kRetV + 8;
    bf16 *kh = reinterpret_cast<bf16*>(rt_sm), *kl = kh + kRetT * kPitch, *vs = kl + kRetT * kPitch;
    const int head = blockIdx.x, chunk = blockIdx.y, chunks = gridDim.y, v0 = blockIdx.z * kRetV, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, c = lane & 3;
    const int t0 = chunk * kRetT, len = min(kRetT, a.tokens - t0), n = a.n, half = a.rot_dims / 2, items = N - half;
    const uint32_t pos0 = seq_position(a.seq, a.pos, 0) + t0;
    decay_powers(a.decay[head], pw);
    __syncthreads();
    const float scale = 1.0f / sqrtf(static_cast<float>(n));
    for (int i = tid; i < kRetT * items; i += 128) {
        const int t = i / items, j = i % items;
        const float* p = a.p + size_t(t0 + min(t, len - 1)) * a.ld + a.heads * n + head * n;
        const float f = t < len ? scale * pw[len - 1 - t] : 0.0f;
        if (j < half) {
            const float2 k = rotate_pair(p[j], p[j + half], rotation(a.turns[j], pos0 + t));
            put_split(kh, kl, t * kPitch + j, k.x * f), put_split(kh, kl, t * kPitch + j + half, k.y * f);
        } else {
            put_split(kh, kl, t * kPitch + j + half, j + half < n ? p[j + half] * f : 0.0f);
        }
    }
    for (int i = tid; i < kRetT * kRetV; i += 128) {
        const int t = i / kRetV, v = i % kRetV;
        vs[t * kVPitch + v] = __float2bfloat16_rn(t < len && v0 + v < a.vdim ? a.p[size_t(t0 + t) * a.ld + 2 * a.heads * n + head * a.vdim + v0 + v] : 0.0f);
    }
    __syncthreads();
    float u[N / 8][4];
#pragma unroll
    for (int j = 0; j < N / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) u[j][e] = 0.0f;
#pragma unroll
    for (int s = 0; s < kRetT / 16; ++s) {
        uint32_t xv[4];
        load_frag_b(xv, vs + s * 16 * kVPitch + warp * 16, kVPitch);
        const uint32_t xt[4] = {xv[0], xv[2], xv[1], xv[3]};  // transposed: an A operand, value columns as rows
#pragma unroll
        for (int j = 0; j < N / 8; j += 2) {
            uint32_t h[4], l[4];
            load_frag_b(h, kh + s * 16 * kPitch + j * 8, kPitch);
            load_frag_b(l, kl + s * 16 * kPitch + j * 8, kPitch);
            mma_16816(u[j], xt, h[0], h[1]), mma_16816(u[j + 1], xt, h[2], h[3]);
            mma_16816(u[j], xt, l[0], l[1]), mma_16816(u[j + 1], xt, l[2], l[3]);
        }
    }
    float* out = r.work.u + ((size_t(head) * chunks + chunk) * r.work.v_pad + v0 + warp * 16) * N;
#pragma unroll
    for (int j = 0; j < N / 8; ++j) {
        *reinterpret_cast<float2*>(out + size_t(g) * N + j * 8 + 2 * c) = make_float2(u[j][0], u[j][1]);
        *reinterpret_cast<float2*>(out + size_t(g + 8) * N + j * 8 + 2 * c) = make_float2(u[j][2], u[j][3]);
    }
}

// The state before every chunk, and after the last one. A thread takes four elements of a head's state. grid: (v_pad * rows / 512, heads)
__global__ void __launch_bounds__(128) retention_carry_kernel(const __grid_constant__ RetentionArgs r) {
    const ScanArgs& a = r.scan;
    const int head = blockIdx.y, chunks = (a.tokens + kRetT - 1) / kRetT, rows = r.work.rows;
    const size_t size = size_t(r.work.v_pad) * rows, at = (size_t(blockIdx.x) * 128 + threadIdx.x) * 4;
    const int v = static_cast<int>(at / rows), d = static_cast<int>(at % rows);
    const uint32_t pos0 = seq_position(a.seq, a.pos, 0);
    const float decay = a.decay[head], whole = decay > 0.0f ? exp2f(static_cast<float>(kRetT) * log2f(decay)) : 0.0f;
    float* state = a.state + (size_t(head) * a.vdim + v) * a.n;
    float s[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) s[e] = pos0 > 0 && v < a.vdim && d + e < a.n ? state[d + e] : 0.0f;
    const float* u = r.work.u + size_t(head) * chunks * size + at;
    bf16 *hi = r.work.s_hi + size_t(head) * chunks * size + at, *lo = r.work.s_lo + size_t(head) * chunks * size + at;
    for (int c0 = 0; c0 < chunks; c0 += 8) {
        float4 b[8];  // eight chunks' loads in flight
#pragma unroll
        for (int k = 0; k < 8; ++k)
            if (c0 + k < chunks) b[k] = *reinterpret_cast<const float4*>(u + (c0 + k) * size);
#pragma unroll
        for (int k = 0; k < 8; ++k)
            if (c0 + k < chunks) {
                uint2 h, l;
                split_bf16(s[0], s[1], &h.x, &l.x), split_bf16(s[2], s[3], &h.y, &l.y);
                *reinterpret_cast<uint2*>(hi + (c0 + k) * size) = h;
                *reinterpret_cast<uint2*>(lo + (c0 + k) * size) = l;
                const int len = min(kRetT, a.tokens - (c0 + k) * kRetT);
                const float f = len == kRetT ? whole : decay > 0.0f ? exp2f(static_cast<float>(len) * log2f(decay)) : 0.0f;
                s[0] = fmaf(f, s[0], b[k].x), s[1] = fmaf(f, s[1], b[k].y), s[2] = fmaf(f, s[2], b[k].z), s[3] = fmaf(f, s[3], b[k].w);
            }
    }
#pragma unroll
    for (int e = 0; e < 4; ++e)
        if (v < a.vdim && d + e < a.n) state[d + e] = s[e];
}

// Outputs of a chunk. grid: (heads, chunks), 128 threads; a warp owns 16 tokens and all value columns
template <int N> __host__ __device__ constexpr size_t retention_out_smem() { return size_t(4 * kRetT) * (N + 8) * 2 + size_t(kRetT) * (kRetV + 8) * 2; }
template <int N, int V>
__global__ void __launch_bounds__(128) retention_out_kernel(const __grid_constant__ RetentionArgs r) {
    extern __shared__ __align__(16) unsigned char rt_sm[];
    __shared__ float pw[kRetT + 1];
    const ScanArgs& a = r.scan;
    constexpr int kPitch = N + 8, kVPitch = kRetV + 8;
    bf16 *qh = reinterpret_cast<bf16*>(rt_sm), *ql = qh + kRetT * kPitch, *kh = ql + kRetT * kPitch, *kl = kh + kRetT * kPitch, *vs = kl + kRetT * kPitch;
    const int head = blockIdx.x, chunk = blockIdx.y, chunks = gridDim.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, c = lane & 3;
    const int t0 = chunk * kRetT, len = min(kRetT, a.tokens - t0), n = a.n, half = a.rot_dims / 2, items = N - half;
    const uint32_t pos0 = seq_position(a.seq, a.pos, 0) + t0;
    decay_powers(a.decay[head], pw);
    const float scale = 1.0f / sqrtf(static_cast<float>(n));
    for (int i = tid; i < kRetT * items; i += 128) {
        const int t = i / items, j = i % items;
        const float* p = a.p + size_t(t0 + min(t, len - 1)) * a.ld + head * n;
        const float* pk = p + a.heads * n;
        const bool there = t < len;
        if (j < half) {
            const float2 cs = rotation(a.turns[j], pos0 + t);
            const float2 q = rotate_pair(p[j], p[j + half], cs), k = rotate_pair(pk[j], pk[j + half], cs);
            put_split(qh, ql, t * kPitch + j, there ? q.x : 0.0f), put_split(qh, ql, t * kPitch + j + half, there ? q.y : 0.0f);
            put_split(kh, kl, t * kPitch + j, there ? k.x * scale : 0.0f), put_split(kh, kl, t * kPitch + j + half, there ? k.y * scale : 0.0f);
        } else {
            const bool in = there && j + half < n;
            put_split(qh, ql, t * kPitch + j + half, in ? p[j + half] : 0.0f);
            put_split(kh, kl, t * kPitch + j + half, in ? pk[j + half] * scale : 0.0f);
        }
    }
    __syncthreads();
    // decayed scores of the chunk's tokens, as A operands of the product with the values
    uint32_t ph[kRetT / 16][4], pl[kRetT / 16][4];
    {
        float s[kRetT / 8][4];
#pragma unroll
        for (int j = 0; j < kRetT / 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) s[j][e] = 0.0f;
#pragma unroll 4
        for (int k = 0; k < N / 16; ++k) {
            uint32_t h[4], l[4];
            load_frag_a(h, qh + warp * 16 * kPitch + k * 16, kPitch), load_frag_a(l, ql + warp * 16 * kPitch + k * 16, kPitch);
#pragma unroll
            for (int j = 0; j < kRetT / 8; j += 2) {
                uint32_t bh[4], bl[4];
                load_frag_bt(bh, kh + j * 8 * kPitch + k * 16, kPitch), load_frag_bt(bl, kl + j * 8 * kPitch + k * 16, kPitch);
                mma_16816(s[j], h, bh[0], bh[1]), mma_16816(s[j + 1], h, bh[2], bh[3]);
                mma_16816(s[j], h, bl[0], bl[1]), mma_16816(s[j + 1], h, bl[2], bl[3]);
                mma_16816(s[j], l, bh[0], bh[1]), mma_16816(s[j + 1], l, bh[2], bh[3]);
            }
        }
#pragma unroll
        for (int j = 0; j < kRetT / 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int back = warp * 16 + g + (e >> 1) * 8 - (j * 8 + 2 * c + (e & 1));
                s[j][e] = back >= 0 ? s[j][e] * pw[max(back, 0)] : 0.0f;
            }
#pragma unroll
        for (int k = 0; k < kRetT / 16; ++k) {
            split_bf16(s[2 * k][0], s[2 * k][1], &ph[k][0], &pl[k][0]), split_bf16(s[2 * k][2], s[2 * k][3], &ph[k][1], &pl[k][1]);
            split_bf16(s[2 * k + 1][0], s[2 * k + 1][1], &ph[k][2], &pl[k][2]), split_bf16(s[2 * k + 1][2], s[2 * k + 1][3], &ph[k][3], &pl[k][3]);
        }
    }
    const float from_state[2] = {pw[warp * 16 + g + 1], pw[warp * 16 + g + 9]};
    bf16 *sh = kh, *sl = kl;  // the keys' place, 64 rows of the state at a time
    float o[V / 8][4], ss[2] = {0.0f, 0.0f};
#pragma unroll
    for (int part = 0; part < V / kRetV; ++part) {
        const int v0 = part * kRetV;
        __syncthreads();
        const size_t at = ((size_t(head) * chunks + chunk) * r.work.v_pad + v0) * N;
        for (int i = tid; i < kRetV * (N / 8); i += 128) {
            const int v = i / (N / 8), p = i % (N / 8);
            cp_async16(sh + v * kPitch + p * 8, r.work.s_hi + at + size_t(v) * N + p * 8, true);
            cp_async16(sl + v * kPitch + p * 8, r.work.s_lo + at + size_t(v) * N + p * 8, true);
        }
        cp_async_commit_group();
        for (int i = tid; i < kRetT * kRetV; i += 128) {
            const int t = i / kRetV, v = i % kRetV;
            vs[t * kVPitch + v] = __float2bfloat16_rn(t < len && v0 + v < a.vdim ? a.p[size_t(t0 + t) * a.ld + 2 * a.heads * n + head * a.vdim + v0 + v] : 0.0f);
        }
        cp_async_wait_group<0>();
        __syncthreads();
        constexpr int kCols = kRetV / 8;
        float (*po)[4] = o + part * kCols;
#pragma unroll
        for (int j = 0; j < kCols; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) po[j][e] = 0.0f;
#pragma unroll 4
        for (int k = 0; k < N / 16; ++k) {
            uint32_t h[4], l[4];
            load_frag_a(h, qh + warp * 16 * kPitch + k * 16, kPitch), load_frag_a(l, ql + warp * 16 * kPitch + k * 16, kPitch);
#pragma unroll
            for (int j = 0; j < kCols; j += 2) {
                uint32_t bh[4], bl[4];
                load_frag_bt(bh, sh + j * 8 * kPitch + k * 16, kPitch), load_frag_bt(bl, sl + j * 8 * kPitch + k * 16, kPitch);
                mma_16816(po[j], h, bh[0], bh[1]), mma_16816(po[j + 1], h, bh[2], bh[3]);
                mma_16816(po[j], h, bl[0], bl[1]), mma_16816(po[j + 1], h, bl[2], bl[3]);
                mma_16816(po[j], l, bh[0], bh[1]), mma_16816(po[j + 1], l, bh[2], bh[3]);
            }
        }
#pragma unroll
        for (int j = 0; j < kCols; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) po[j][e] *= from_state[e >> 1];
#pragma unroll
        for (int k = 0; k < kRetT / 16; ++k)
#pragma unroll
            for (int j = 0; j < kCols; j += 2) {
                uint32_t b[4];
                load_frag_b(b, vs + k * 16 * kVPitch + j * 8, kVPitch);
                mma_16816(po[j], ph[k], b[0], b[1]), mma_16816(po[j + 1], ph[k], b[2], b[3]);
                mma_16816(po[j], pl[k], b[0], b[1]), mma_16816(po[j + 1], pl[k], b[2], b[3]);
            }
#pragma unroll
        for (int j = 0; j < kCols; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) ss[e >> 1] = fmaf(po[j][e], po[j][e], ss[e >> 1]);  // (columns beyond vdim are zero)
    }
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        ss[h] += __shfl_xor_sync(0xffffffffu, ss[h], 1);
        ss[h] += __shfl_xor_sync(0xffffffffu, ss[h], 2);
        const int t = warp * 16 + g + 8 * h;
        if (t >= len) continue;
        const float inv = 1.0f / sqrtf(ss[h] / static_cast<float>(a.vdim) + r.eps);
        const float* gate = a.p + size_t(t0 + t) * a.ld + 2 * a.heads * n + a.heads * a.vdim + head * a.vdim;
        bf16* out = static_cast<bf16*>(r.out) + size_t(t0 + t) * r.out_pitch + head * a.vdim;
#pragma unroll
        for (int j = 0; j < V / 8; ++j)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int v = j * 8 + 2 * c + e;
                if (v < a.vdim) out[v] = __float2bfloat16_rn(o[j][2 * h + e] * inv * silu_f(gate[v]));
            }
    }
}

}  // namespace qtb
