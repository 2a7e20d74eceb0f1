// Retention (gated_scan.cuh) over many tokens. With one decay a per head the state after a chunk of T tokens is a^T S + U, where U depends on the
// chunk's own keys and values only, and
//
//   y_t = a^(t + 1) q_t S + sum over s <= t of a^(t - s) (q_t . k_s) v_s        t, s: places in the chunk
//
// so the chunks need not follow one another: U of every chunk at once, then S at every chunk's start (one multiply-add per element and chunk), then
// every chunk's outputs at once. 64 tokens a chunk, products on the warp tensor cores; queries, keys, states and decayed weights or values go in as
// two bf16 terms. The last kernel also divides each head's output by its root mean square and multiplies it by silu(g).
#pragma once
#include "gated_scan.cuh"
#include "mma_bf16.cuh"

namespace qtb {

constexpr int kRetT = 64;      // tokens of a chunk
constexpr int kRetV = 64;      // value columns per block of the state kernel
constexpr int kRetPart = 32;   // value columns per turn of the output kernel
constexpr int kRetPrep = 8;    // tokens per block of the preparing kernel
constexpr int kRetStages = 3;

// Compiled sizes: rows of the state and value columns, 0 if a head is too large.
inline int retention_rows(int dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : dim <= 128 ? 128 : dim <= 256 ? 256 : 0; }
inline int retention_cols(int vdim) { return vdim <= 64 ? 64 : vdim <= 128 ? 128 : vdim <= 256 ? 256 : 0; }
inline int retention_chunks(int tokens) { return (tokens + kRetT - 1) / kRetT; }

struct RetentionWork {
    bf16 *q_hi, *q_lo, *k_hi, *k_lo;  // rotated (keys also scaled), [head][token][rows], zero beyond dim and beyond the last token
    bf16* v;               // [head][token][v_pad]
    float* u;              // [head][chunk][v_pad][rows]
    bf16 *s_hi, *s_lo;     // the state before each chunk, same order
    int rows, v_pad, tokens;  // tokens: rounded up to whole chunks
};
inline size_t retention_work(char* base, int heads, int dim, int vdim, int tokens, RetentionWork* w) {
    w->rows = retention_rows(dim), w->v_pad = retention_cols(vdim), w->tokens = retention_chunks(tokens) * kRetT;
    const size_t n = size_t(heads) * retention_chunks(tokens) * w->v_pad * w->rows, qk = size_t(heads) * w->tokens * w->rows, v = size_t(heads) * w->tokens * w->v_pad;
    w->u = reinterpret_cast<float*>(base), w->s_hi = reinterpret_cast<bf16*>(w->u + n), w->s_lo = w->s_hi + n;
    w->q_hi = w->s_lo + n, w->q_lo = w->q_hi + qk, w->k_hi = w->q_lo + qk, w->k_lo = w->k_hi + qk, w->v = w->k_lo + qk;
    return n * 8 + qk * 8 + v * 2;
}

struct RetentionArgs {
    ScanArgs scan;
    RetentionWork work;
    float eps;             // of the heads' norm
    void* out;             // [token][out_pitch], bf16
    int out_pitch;
    bool pairs;            // sizes and columns are even: two neighbouring elements at a time
};

// powers a^0 .. a^T of a head's decay
__device__ __forceinline__ void decay_powers(float decay, float* pw) {
    for (int i = threadIdx.x; i <= kRetT; i += blockDim.x) pw[i] = i == 0 ? 1.0f : decay > 0.0f ? exp2f(static_cast<float>(i) * log2f(decay)) : 0.0f;
}
// Queries, keys and values of every token as the products take them. PAIRS: two neighbouring elements at a time (even sizes and columns).
// Four heads a block: they share the angles. grid: (ceil(heads / 4), padded tokens / 8), 256 threads
template <bool PAIRS>
__global__ void __launch_bounds__(256) retention_prepare_kernel(const __grid_constant__ RetentionArgs r) {
    __shared__ float2 angle[kRetPrep][128];  // (a head has at most 256 rotated dimensions)
    const ScanArgs& a = r.scan;
    const RetentionWork& w = r.work;
    constexpr int S = PAIRS ? 2 : 1;
    const int t0 = blockIdx.y * kRetPrep, tid = threadIdx.x, n = a.n, half = a.rot_dims / 2, head0 = blockIdx.x * 4, heads = min(4, a.heads - head0);
    const uint32_t pos0 = seq_position(a.seq, a.pos, 0);
    const float scale = 1.0f / sqrtf(static_cast<float>(n));
    for (int i = tid; i < kRetPrep * half; i += 256) angle[i / half][i % half] = rotation(a.turns[i % half], pos0 + t0 + i / half);
    __syncthreads();
    auto put = [&](bf16* hi, bf16* lo, size_t at, const float (&v)[S]) {
        if constexpr (PAIRS) {
            uint32_t h, l;
            split_bf16(v[0], v[1], &h, &l);
            *reinterpret_cast<uint32_t*>(hi + at) = h, *reinterpret_cast<uint32_t*>(lo + at) = l;
        } else {
            const bf16 h = __float2bfloat16_rn(v[0]);
            hi[at] = h, lo[at] = __float2bfloat16_rn(v[0] - __bfloat162float(h));
        }
    };
    auto get = [&](const float* p, bool there, float (&v)[S]) {
        if constexpr (PAIRS) {
            const float2 f = there ? __ldg(reinterpret_cast<const float2*>(p)) : make_float2(0.0f, 0.0f);
            v[0] = f.x, v[1] = f.y;
        } else {
            v[0] = there ? __ldg(p) : 0.0f;
        }
    };
    const int items = (w.rows - half) / S, cols = w.v_pad / S;  // an item is a pair to rotate (two neighbouring ones), or elements that stay as they are
#pragma unroll 4
    for (int i = tid; i < heads * kRetPrep * items; i += 256) {
        const int row = i / items, j = i % items * S, head = head0 + row / kRetPrep, t = t0 + row % kRetPrep;
        const bool there = t < a.tokens;
        const float* p = a.p + size_t(min(t, a.tokens - 1)) * a.ld + head * n;
        const float* pk = p + a.heads * n;
        const size_t at = (size_t(head) * w.tokens + t) * w.rows;
        const bool turns = j < half, in = there && j + half < n;  // (a rotated pair's second element is below n)
        float q[S], k[S], q2[S], k2[S];
        get(p + j, there && turns, q), get(p + j + half, in, q2), get(pk + j, there && turns, k), get(pk + j + half, in, k2);
#pragma unroll
        for (int e = 0; e < S; ++e) {
            if (turns) {
                const float2 cs = angle[t - t0][j + e];
                const float2 rq = rotate_pair(q[e], q2[e], cs), rk = rotate_pair(k[e], k2[e], cs);
                q[e] = rq.x, q2[e] = rq.y, k[e] = rk.x, k2[e] = rk.y;
            }
            k[e] *= scale, k2[e] *= scale;
        }
        if (turns) put(w.q_hi, w.q_lo, at + j, q), put(w.k_hi, w.k_lo, at + j, k);
        put(w.q_hi, w.q_lo, at + j + half, q2), put(w.k_hi, w.k_lo, at + j + half, k2);
    }
#pragma unroll 4
    for (int i = tid; i < heads * kRetPrep * cols; i += 256) {
        const int row = i / cols, c = i % cols * S, head = head0 + row / kRetPrep, t = t0 + row % kRetPrep;
        float v[S];
        get(a.p + size_t(min(t, a.tokens - 1)) * a.ld + 2 * a.heads * n + head * a.vdim + c, t < a.tokens && c < a.vdim, v);
        bf16* out = w.v + (size_t(head) * w.tokens + t) * w.v_pad + c;
        if constexpr (PAIRS) *reinterpret_cast<uint32_t*>(out) = pack_bf16(v[0], v[1]);
        else *out = __float2bfloat16_rn(v[0]);
    }
}

// U of every chunk. grid: (heads, chunks, v_pad / 64), 128 threads; a warp owns 16 value columns
template <int N> __host__ __device__ constexpr size_t retention_state_smem() { return size_t(2 * kRetT) * (N + 8) * 2 + size_t(kRetT) * (kRetV + 8) * 2; }
template <int N>
__global__ void __launch_bounds__(128) retention_state_kernel(const __grid_constant__ RetentionArgs r) {
    extern __shared__ __align__(16) unsigned char rt_sm[];
    __shared__ float pw[kRetT + 1];
    const ScanArgs& a = r.scan;
    constexpr int kPitch = N + 8, kVPitch = kRetV + 8;
    bf16 *kh = reinterpret_cast<bf16*>(rt_sm), *kl = kh + kRetT * kPitch, *vs = kl + kRetT * kPitch;
    const int head = blockIdx.x, chunk = blockIdx.y, chunks = gridDim.y, v0 = blockIdx.z * kRetV, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, c = lane & 3;
    const int t0 = chunk * kRetT, len = min(kRetT, a.tokens - t0);
    const size_t row0 = size_t(head) * r.work.tokens + t0;
    for (int i = tid; i < kRetT * (N / 8); i += 128) {
        const int t = i / (N / 8), p = i % (N / 8);
        cp_async16(kh + t * kPitch + p * 8, r.work.k_hi + (row0 + t) * N + p * 8, true);
        cp_async16(kl + t * kPitch + p * 8, r.work.k_lo + (row0 + t) * N + p * 8, true);
    }
    for (int i = tid; i < kRetT * (kRetV / 8); i += 128) {
        const int t = i / (kRetV / 8), p = i % (kRetV / 8);
        cp_async16(vs + t * kVPitch + p * 8, r.work.v + (row0 + t) * r.work.v_pad + v0 + p * 8, true);
    }
    cp_async_commit_group();
    decay_powers(a.decay[head], pw);
    cp_async_wait_group<0>();
    __syncthreads();
    float u[N / 8][4];
#pragma unroll
    for (int j = 0; j < N / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) u[j][e] = 0.0f;
#pragma unroll
    for (int s = 0; s < kRetT / 16; ++s) {
        uint32_t xv[4], xh[4], xl[4];
        load_frag_b(xv, vs + s * 16 * kVPitch + warp * 16, kVPitch);
#pragma unroll
        for (int e = 0; e < 4; ++e) {  // transposed an A operand, value columns as rows; its tokens: s * 16 + 2 c, + 1 (e < 2), + 8, + 9
            const uint32_t x = xv[((e & 1) << 1) | (e >> 1)];
            const int t = s * 16 + 2 * c + (e >> 1) * 8;  // (tokens beyond len: keys and values are zero)
            split_bf16(__uint_as_float(x << 16) * pw[max(len - 1 - t, 0)], __uint_as_float(x & 0xffff0000u) * pw[max(len - 2 - t, 0)], &xh[e], &xl[e]);
        }
#pragma unroll
        for (int j = 0; j < N / 8; j += 2) {
            uint32_t h[4], l[4];
            load_frag_b(h, kh + s * 16 * kPitch + j * 8, kPitch);
            load_frag_b(l, kl + s * 16 * kPitch + j * 8, kPitch);
            mma_16816(u[j], xh, h[0], h[1]), mma_16816(u[j + 1], xh, h[2], h[3]);
            mma_16816(u[j], xl, h[0], h[1]), mma_16816(u[j + 1], xl, h[2], h[3]);
            mma_16816(u[j], xh, l[0], l[1]), mma_16816(u[j + 1], xh, l[2], l[3]);
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

// Outputs of a chunk. grid: (heads, chunks), 128 threads; a warp owns 16 tokens and all value columns, 32 of them at a time: the next 64 columns of
// the state and the values are on their way while the products of these are made.
template <int N> __host__ __device__ constexpr size_t retention_out_stage() { return size_t(2 * kRetPart) * (N + 8) * 2 + size_t(kRetT) * (kRetPart + 8) * 2; }
template <int N> __host__ __device__ constexpr size_t retention_out_smem() { return size_t(2 * kRetT) * (N + 8) * 2 + kRetStages * retention_out_stage<N>(); }
template <int N, int V>
__global__ void __launch_bounds__(128) retention_out_kernel(const __grid_constant__ RetentionArgs r) {
    extern __shared__ __align__(16) unsigned char rt_sm[];
    __shared__ float pw[kRetT + 1];
    const ScanArgs& a = r.scan;
    constexpr int kPitch = N + 8, kVPitch = kRetPart + 8, kParts = V / kRetPart, kCols = kRetPart / 8;
    constexpr size_t kStage = retention_out_stage<N>();
    static_assert((kRetStages - 1) * kStage >= size_t(2 * kRetT) * kPitch * 2, "the keys fit the stages behind the first until the scores are made");
    bf16 *qh = reinterpret_cast<bf16*>(rt_sm), *ql = qh + kRetT * kPitch;
    unsigned char* stages = reinterpret_cast<unsigned char*>(ql + kRetT * kPitch);
    bf16 *kh = reinterpret_cast<bf16*>(stages + kStage), *kl = kh + kRetT * kPitch;
    const int head = blockIdx.x, chunk = blockIdx.y, chunks = gridDim.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, c = lane & 3;
    const int t0 = chunk * kRetT, len = min(kRetT, a.tokens - t0), n = a.n;
    const size_t row0 = size_t(head) * r.work.tokens + t0;
    for (int i = tid; i < kRetT * (N / 8); i += 128) {
        const int t = i / (N / 8), p = i % (N / 8), at = t * kPitch + p * 8;
        const size_t from = (row0 + t) * N + p * 8;
        cp_async16(qh + at, r.work.q_hi + from, true), cp_async16(ql + at, r.work.q_lo + from, true);
        cp_async16(kh + at, r.work.k_hi + from, true), cp_async16(kl + at, r.work.k_lo + from, true);
    }
    cp_async_commit_group();
    auto fetch = [&](int part) {
        if (part >= kParts) {
            cp_async_commit_group();  // (an empty group keeps the count of groups in step with the parts)
            return;
        }
        bf16 *sh = reinterpret_cast<bf16*>(stages + (part % kRetStages) * kStage), *sl = sh + kRetPart * kPitch, *vs = sl + kRetPart * kPitch;
        const size_t at = ((size_t(head) * chunks + chunk) * r.work.v_pad + part * kRetPart) * N;
        for (int i = tid; i < kRetPart * (N / 8); i += 128) {
            const int v = i / (N / 8), p = i % (N / 8);
            cp_async16(sh + v * kPitch + p * 8, r.work.s_hi + at + size_t(v) * N + p * 8, true);
            cp_async16(sl + v * kPitch + p * 8, r.work.s_lo + at + size_t(v) * N + p * 8, true);
        }
        for (int i = tid; i < kRetT * (kRetPart / 8); i += 128) {
            const int t = i / (kRetPart / 8), p = i % (kRetPart / 8);
            cp_async16(vs + t * kVPitch + p * 8, r.work.v + (row0 + t) * r.work.v_pad + part * kRetPart + p * 8, true);
        }
        cp_async_commit_group();
    };
    fetch(0);
    decay_powers(a.decay[head], pw);
    cp_async_wait_group<1>();
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
                if (j / 2 > warp) continue;  // (all of these keys come later)
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
    __syncthreads();  // every warp is done with the keys
    fetch(1);
    float o[V / 8][4], ss[2] = {0.0f, 0.0f};
#pragma unroll
    for (int part = 0; part < kParts; ++part) {
        cp_async_wait_group<1>();
        __syncthreads();
        fetch(part + 2);  // into the stage of the part before this one, which every warp has left
        const bf16 *sh = reinterpret_cast<const bf16*>(stages + (part % kRetStages) * kStage), *sl = sh + kRetPart * kPitch, *vs = sl + kRetPart * kPitch;
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
        for (int k = 0; k < kRetT / 16; ++k) {
            if (k > warp) continue;  // (their weights are zero)
#pragma unroll
            for (int j = 0; j < kCols; j += 2) {
                uint32_t b[4];
                load_frag_b(b, vs + k * 16 * kVPitch + j * 8, kVPitch);
                mma_16816(po[j], ph[k], b[0], b[1]), mma_16816(po[j + 1], ph[k], b[2], b[3]);
                mma_16816(po[j], pl[k], b[0], b[1]), mma_16816(po[j + 1], pl[k], b[2], b[3]);
            }
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
        const auto gated = [&](float v, float z) { return v * inv * __fdividef(z, 1.0f + __expf(-z)); };
        if (r.pairs) {
#pragma unroll
            for (int j0 = 0; j0 < V / 8; j0 += 8) {
                float2 z[8];  // eight loads in flight
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    const int v = (j0 + j) * 8 + 2 * c;
                    z[j] = v < a.vdim ? __ldg(reinterpret_cast<const float2*>(gate + v)) : make_float2(0.0f, 0.0f);
                }
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    const int v = (j0 + j) * 8 + 2 * c;
                    if (v < a.vdim) *reinterpret_cast<uint32_t*>(out + v) = pack_bf16(gated(o[j0 + j][2 * h], z[j].x), gated(o[j0 + j][2 * h + 1], z[j].y));
                }
            }
            continue;
        }
#pragma unroll
        for (int j = 0; j < V / 8; ++j)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int v = j * 8 + 2 * c + e;
                if (v < a.vdim) out[v] = __float2bfloat16_rn(gated(o[j][2 * h + e], __ldg(gate + v)));
            }
    }
}

}  // namespace qtb
