// The recurrences of gated_scan.cuh over many tokens, 16 at a time:
//
//   y_t = (q_t (.) F_t) S_0 + sum over s <= t of A_ts x_s        A_ts = sum over rows d of q_t k_s prod_{s < r <= t} a_r
//   S_16 = F_16 (.) S_0 + sum over s of (k_s (.) prod_{s < r} a_r) x_s^T       F_t = a_1 ... a_t
//
// What does not depend on the state is made for all chunks at once: for mamba2 the convolution, the steps dt with the running sums of their
// log decays, and the products C B^T (the decays are numbers, so A and the scaled operands follow from them inside the scan); for hgrn2, where
// every row decays on its own, A (running products in 32-bit, nothing is divided), q (.) F and k (.) rest as two bf16 terms each, and F_16. The
// scan then walks the chunks of a head with the state in the registers of its products: a warp owns 16 columns, the state transposed, so that
// the sums of one product are, rounded to hi + lo terms, an operand of the next. Inputs of the next chunk are fetched while one is computed.
#pragma once
#include "gated_scan.cuh"
#include "mma_bf16.cuh"

namespace qtb {

constexpr int kChunkT = 16, kChunkV = 64;  // tokens of a chunk; state columns of a block (16 per warp)
constexpr int kChunkStages = 4;             // chunks whose inputs are in shared memory or on the way

// Row count of the state the scan is compiled for, 0 if it is too large for it.
inline int chunk_scan_rows(int n) { return n <= 32 ? 32 : n <= 64 ? 64 : n <= 128 ? 128 : 0; }
inline int chunk_count(int tokens) { return (tokens + kChunkT - 1) / kChunkT; }

// Work space of one layer (bytes from the start of a buffer), tokens rounded up to whole chunks.
struct ChunkWork {
    bf16* xs;      // [token][heads][v_pad]: x, zero beyond vdim and beyond the last token
    bf16* bc;      // mamba2: [token][B, C][groups][rows]
    float* gram;   // mamba2: [chunk][group][16][16] = C B^T
    float* dt;     // mamba2: [head][chunk][dt 16 | running sum of -exp(A_log) dt 16]
    bf16* qk;      // hgrn2: [head][chunk][q hi, q lo, k hi, k lo][16][rows]
    float* a;      // hgrn2: [head][chunk][16][16]
    float* fe;     // hgrn2: [head][chunk][rows]
    int v_pad, rows;
};
inline size_t chunk_work(char* base, bool mamba, int heads, int vdim, int n, int groups, int tokens, ChunkWork* w) {
    const size_t t = size_t(chunk_count(tokens)) * kChunkT, c = chunk_count(tokens);
    size_t at = 0;
    auto take = [&](size_t bytes) {
        char* p = base + at;
        at += (bytes + 255) / 256 * 256;
        return p;
    };
    *w = ChunkWork{};
    w->v_pad = (vdim + kChunkV - 1) / kChunkV * kChunkV, w->rows = chunk_scan_rows(n);
    w->xs = reinterpret_cast<bf16*>(take(t * heads * w->v_pad * 2));
    if (mamba) {
        w->bc = reinterpret_cast<bf16*>(take(t * 2 * groups * w->rows * 2));
        w->gram = reinterpret_cast<float*>(take(c * groups * 256 * 4));
        w->dt = reinterpret_cast<float*>(take(c * heads * 32 * 4));
    } else {
        w->qk = reinterpret_cast<bf16*>(take(c * heads * 64 * w->rows * 2));
        w->a = reinterpret_cast<float*>(take(c * heads * 256 * 4));
        w->fe = reinterpret_cast<float*>(take(c * heads * w->rows * 4));
    }
    return at;
}

// mamba2: convolution and silu of every channel into xs and bc. grid: (padded channels / 128, chunks); a thread takes a channel of 16 tokens.
// TAPS: taps of the convolution where they are few enough to keep their inputs in registers, 0 for any number.
template <int TAPS>
__global__ void __launch_bounds__(128) ssd_conv_kernel(const __grid_constant__ ScanArgs a, const __grid_constant__ ChunkWork w) {
    const int c = blockIdx.x * 128 + threadIdx.x, nx = a.heads * w.v_pad, nbc = 2 * a.groups * w.rows, inner = a.heads * a.vdim, channels = inner + 2 * a.groups * a.n;
    if (c >= nx + nbc) return;
    int real = -1;  // the channel of the convolution, -1: padding
    if (c < nx) {
        if (c % w.v_pad < a.vdim) real = c / w.v_pad * a.vdim + c % w.v_pad;
    } else if ((c - nx) % w.rows < a.n) {
        real = inner + (c - nx) / w.rows * a.n + (c - nx) % w.rows;
    }
    bf16* out = c < nx ? w.xs + c : w.bc + (c - nx);
    const size_t step = c < nx ? nx : nbc;
    const uint32_t pos0 = seq_position(a.seq, a.pos, 0);
    const float* ring = a.conv;
    const int t0 = blockIdx.y * kChunkT;
    if (TAPS > 0) {
        constexpr int kBack = TAPS > 0 ? TAPS - 1 : 0;
        float u[kChunkT + kBack], wt[TAPS > 0 ? TAPS : 1];
        const int c0 = max(real, 0);
        const float bias = a.conv_b[c0];
#pragma unroll
        for (int k = 0; k < TAPS; ++k) wt[k] = a.conv_w[size_t(c0) * TAPS + k];
#pragma unroll
        for (int i = 0; i < kChunkT + kBack; ++i) {  // all inputs in flight
            const int t = t0 + i - kBack;
            const bool there = real >= 0 && t < a.tokens && static_cast<int>(pos0) + t >= 0;
            const float* src = t >= 0 ? a.p + size_t(t) * a.ld + inner + c0 : ring + size_t((pos0 + t) % TAPS) * channels + c0;
            u[i] = there ? *src : 0.0f;
        }
#pragma unroll
        for (int i = 0; i < kChunkT; ++i) {
            float s = bias;
#pragma unroll
            for (int k = 0; k < TAPS; ++k) s = fmaf(wt[k], u[i + k], s);
            out[size_t(t0 + i) * step] = __float2bfloat16_rn(real >= 0 && t0 + i < a.tokens ? silu_f(s) : 0.0f);
        }
        return;
    }
    for (int i = 0; i < kChunkT; ++i) {
        const int t = t0 + i;
        out[size_t(t) * step] = __float2bfloat16_rn(real >= 0 && t < a.tokens ? conv_silu(a, ring, t, t, pos0 + t, real, channels, inner) : 0.0f);
    }
}

// mamba2: per chunk the products of C and B (blocks x < groups), and per head dt and the running sums of the log decays (the last block).
// grid: (groups + 1, chunks), 256 threads
__global__ void __launch_bounds__(256) ssd_gram_kernel(const __grid_constant__ ScanArgs a, const __grid_constant__ ChunkWork w) {
    const int g = blockIdx.x, chunk = blockIdx.y, chunks = gridDim.y, tid = threadIdx.x;
    if (g == a.groups) {
        const int inner = a.heads * a.vdim, col = 2 * inner + 2 * a.groups * a.n;
        for (int h = tid; h < a.heads; h += 256) {
            float* out = w.dt + (size_t(h) * chunks + chunk) * 32;
            const float rate = -expf(a.a_log[h]), bias = a.dt_bias[h];
            float sum = 0.0f;
            for (int i = 0; i < kChunkT; ++i) {
                const int t = chunk * kChunkT + i;
                const float dt = t < a.tokens ? softplus_f(a.p[size_t(t) * a.ld + col + h] + bias) : 0.0f;
                sum += rate * dt;
                out[i] = dt, out[16 + i] = sum;
            }
        }
        return;
    }
    extern __shared__ float gram_sm[];  // C rows, then B rows
    const int pitch = w.rows + 1;
    for (int i = tid; i < 2 * kChunkT * w.rows; i += 256) {
        const int which = i / (kChunkT * w.rows), t = i / w.rows % kChunkT, d = i % w.rows;
        gram_sm[(which * kChunkT + t) * pitch + d] = __bfloat162float(w.bc[((size_t(chunk * kChunkT + t) * 2 + (1 - which)) * a.groups + g) * w.rows + d]);
    }
    __syncthreads();
    const float *c = gram_sm + (tid >> 4) * pitch, *b = gram_sm + (kChunkT + (tid & 15)) * pitch;
    float s = 0.0f;
    for (int d = 0; d < w.rows; ++d) s = fmaf(c[d], b[d], s);
    w.gram[(size_t(chunk) * a.groups + g) * 256 + tid] = s;
}

// hgrn2: gates, A, scaled operands. grid: (heads, chunks), 128 threads; n <= ROWS
template <int ROWS>
__global__ void __launch_bounds__(128) hgrn_prep_kernel(const __grid_constant__ ScanArgs a, const __grid_constant__ ChunkWork w) {
    extern __shared__ float prep_sm[];
    const int head = blockIdx.x, chunk = blockIdx.y, chunks = gridDim.y, tid = threadIdx.x, n = a.n;
    constexpr int rows = ROWS;
    float *q = prep_sm, *k = q + kChunkT * rows, *f = k + kChunkT * rows;
    for (int i0 = tid; i0 < kChunkT * rows; i0 += 128 * 4) {  // four elements' loads in flight (kChunkT * rows is a multiple of 512)
        float qr[4], fr[4], low[4];
        bool there[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int i = i0 + 128 * j, t = chunk * kChunkT + i / rows, d = i % rows, c = head * n + min(d, n - 1);
            there[j] = t < a.tokens && d < n;
            const float* p = a.p + size_t(min(t, a.tokens - 1)) * a.ld + c;
            qr[j] = p[0], fr[j] = p[a.heads * n] + a.f_bias[c], low[j] = a.lower[c];
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int i = i0 + 128 * j;
            const float e = expf(-fabsf(fr[j])), r = 1.0f / (1.0f + e), up = fr[j] >= 0.0f ? r : e * r, down = fr[j] >= 0.0f ? e * r : r;  // sigmoids of z and -z
            q[i] = there[j] ? silu_f(qr[j]) : 0.0f;
            f[i] = there[j] ? low[j] + (1.0f - low[j]) * up : 1.0f;
            k[i] = there[j] ? (1.0f - low[j]) * down : 0.0f;
        }
    }
    for (int i0 = tid; i0 < kChunkT * w.v_pad; i0 += 128 * 8) {  // (v_pad is a multiple of 64: whole turns of 1024)
        float v[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const int i = i0 + 128 * j, t = chunk * kChunkT + i / w.v_pad, e = i - (t - chunk * kChunkT) * w.v_pad;
            v[j] = t < a.tokens && e < a.vdim ? a.p[size_t(t) * a.ld + 2 * a.heads * n + head * a.vdim + e] : 0.0f;
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const int i = i0 + 128 * j, t = chunk * kChunkT + i / w.v_pad, e = i - (t - chunk * kChunkT) * w.v_pad;
            w.xs[(size_t(t) * a.heads + head) * w.v_pad + e] = __float2bfloat16_rn(v[j]);
        }
    }
    __syncthreads();
    const size_t at = size_t(head) * chunks + chunk;
    bf16* qk = w.qk + at * 64 * rows;
    auto put = [&](int which, int t, int d, float v) {
        const bf16 hi = __float2bfloat16_rn(v);
        qk[((which)*kChunkT + t) * rows + d] = hi;
        qk[((which + 1) * kChunkT + t) * rows + d] = __float2bfloat16_rn(v - __bfloat162float(hi));
    };
    for (int d = tid; d < rows; d += 128) {
        float prod = 1.0f;
        for (int t = 0; t < kChunkT; ++t) {
            prod *= f[t * rows + d];
            put(0, t, d, q[t * rows + d] * prod);
        }
        w.fe[at * rows + d] = prod;
        float rest = 1.0f;
        for (int t = kChunkT - 1; t >= 0; --t) {
            put(2, t, d, k[t * rows + d] * rest);
            rest *= f[t * rows + d];
        }
    }
    const int s = tid >> 3, dg = tid & 7;  // A: a thread takes a column s and every eighth row of the state
    float acc[kChunkT];
#pragma unroll
    for (int t = 0; t < kChunkT; ++t) acc[t] = 0.0f;
    for (int d = dg; d < n; d += 8) {
        float r = k[s * rows + d];
#pragma unroll
        for (int t = 0; t < kChunkT; ++t) {
            if (t > s) r *= f[t * rows + d];
            if (t >= s) acc[t] = fmaf(q[t * rows + d], r, acc[t]);
        }
    }
#pragma unroll
    for (int t = 0; t < kChunkT; ++t) {
        float v = acc[t];
        v += __shfl_xor_sync(0xffffffffu, v, 1), v += __shfl_xor_sync(0xffffffffu, v, 2), v += __shfl_xor_sync(0xffffffffu, v, 4);
        if (dg == 0) w.a[at * 256 + t * 16 + s] = v;
    }
}

template <int KIND> inline size_t chunk_scan_smem(int rows) {
    const size_t stage = size_t(KIND == kScanMamba2 ? 2 : 4) * kChunkT * (rows + 8) * 2 + size_t(kChunkT) * (kChunkV + 8) * 2 + 256 * 4 + (KIND == kScanMamba2 ? 32 : rows) * 4;
    return kChunkStages * stage;
}

// grid: (heads, ceil(vdim / 64)); warp w owns the state columns 16 w .. 16 w + 15 of the block's 64. y: without mamba2's silu(z), which the
// kernel that norms y applies.
template <int KIND, int ROWS>
__global__ void __launch_bounds__(128) chunk_scan_kernel(const __grid_constant__ ScanArgs a, const __grid_constant__ ChunkWork w) {
    extern __shared__ __align__(16) unsigned char cs_sm[];
    constexpr int kOps = KIND == kScanMamba2 ? 2 : 4, kPitch = ROWS + 8, kVPitch = kChunkV + 8, kTail = KIND == kScanMamba2 ? 32 : ROWS;
    constexpr size_t kStage = size_t(kOps) * kChunkT * kPitch * 2 + size_t(kChunkT) * kVPitch * 2 + 256 * 4 + kTail * 4;
    const int head = blockIdx.x, v0 = blockIdx.y * kChunkV, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, c = lane & 3;
    const int chunks = (a.tokens + kChunkT - 1) / kChunkT, inner = a.heads * a.vdim, group = KIND == kScanMamba2 ? head / (a.heads / a.groups) : 0;
    const uint32_t pos0 = seq_position(a.seq, a.pos, 0);
    const int vw = v0 + warp * 16;
    float* state = a.state + size_t(head) * a.vdim * a.n;
    float S[ROWS / 8][4];
#pragma unroll
    for (int j = 0; j < ROWS / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int v = vw + g + (e >> 1) * 8, d = 8 * j + 2 * c + (e & 1);
            S[j][e] = pos0 > 0 && v < a.vdim && d < a.n ? state[size_t(v) * a.n + d] : 0.0f;
        }
    auto fetch = [&](int chunk) {
        if (chunk >= chunks) {
            cp_async_commit_group();  // (an empty group keeps the count of groups in step with the chunks)
            return;
        }
        unsigned char* st = cs_sm + (chunk % kChunkStages) * kStage;
        bf16* ops = reinterpret_cast<bf16*>(st);
        bf16* xs = ops + kOps * kChunkT * kPitch;
        float* mat = reinterpret_cast<float*>(xs + kChunkT * kVPitch);
        constexpr int kVec = ROWS / 8;
        for (int i = tid; i < kOps * kChunkT * kVec; i += 128) {
            const int op = i / (kChunkT * kVec), t = i / kVec % kChunkT, p = i % kVec;
            const bf16* src = KIND == kScanMamba2 ? w.bc + ((size_t(chunk * kChunkT + t) * 2 + (1 - op)) * a.groups + group) * ROWS + p * 8
                                                  : w.qk + ((size_t(head) * chunks + chunk) * 64 + op * kChunkT + t) * ROWS + p * 8;
            cp_async16(ops + (op * kChunkT + t) * kPitch + p * 8, src, true);
        }
        for (int i = tid; i < kChunkT * (kChunkV / 8); i += 128) {
            const int t = i / (kChunkV / 8), p = i % (kChunkV / 8);
            cp_async16(xs + t * kVPitch + p * 8, w.xs + (size_t(chunk * kChunkT + t) * a.heads + head) * w.v_pad + v0 + p * 8, true);
        }
        const float* m = KIND == kScanMamba2 ? w.gram + (size_t(chunk) * a.groups + group) * 256 : w.a + (size_t(head) * chunks + chunk) * 256;
        const float* tail = KIND == kScanMamba2 ? w.dt + (size_t(head) * chunks + chunk) * 32 : w.fe + (size_t(head) * chunks + chunk) * ROWS;
        for (int i = tid; i < 64 + kTail / 4; i += 128) cp_async16(mat + i * 4, i < 64 ? m + i * 4 : tail + (i - 64) * 4, true);
        cp_async_commit_group();
    };
    for (int i = 0; i < kChunkStages - 1; ++i) fetch(i);
    for (int chunk = 0; chunk < chunks; ++chunk) {
        unsigned char* st = cs_sm + (chunk % kChunkStages) * kStage;
        cp_async_wait_group<kChunkStages - 2>();
        __syncthreads();
        fetch(chunk + kChunkStages - 1);  // into the stage of the chunk before this one, which every warp has left
        if (vw < a.vdim) {
            const bf16* ops = reinterpret_cast<const bf16*>(st);
            const bf16* xs = ops + kOps * kChunkT * kPitch;
            const float* mat = reinterpret_cast<const float*>(xs + kChunkT * kVPitch);
            const float* tail = mat + 256;  // mamba2: dt, running sums; hgrn2: F_16
            uint32_t xv[4];                 // x as a B operand: columns 0..7 (0, 1) and 8..15 (2, 3); transposed it is the A operand {0, 2, 1, 3}
            load_frag_b(xv, xs + warp * 16, kVPitch);
            float O[2][4] = {}, P[3][2][4] = {};  // independent sums: a product waits for the one before it in the same registers
#pragma unroll
            for (int ks = 0; ks < ROWS / 16; ++ks) {
                uint32_t q[4], ql[4], h[4], l[4];
                load_frag_a(q, ops + ks * 16, kPitch);
                split_bf16(S[2 * ks][0], S[2 * ks][1], &h[0], &l[0]), split_bf16(S[2 * ks + 1][0], S[2 * ks + 1][1], &h[1], &l[1]);
                split_bf16(S[2 * ks][2], S[2 * ks][3], &h[2], &l[2]), split_bf16(S[2 * ks + 1][2], S[2 * ks + 1][3], &h[3], &l[3]);
                if (ks & 1) mma_16816(P[0][0], q, h[0], h[1]), mma_16816(P[0][1], q, h[2], h[3]);
                else mma_16816(O[0], q, h[0], h[1]), mma_16816(O[1], q, h[2], h[3]);
                mma_16816(P[1][0], q, l[0], l[1]), mma_16816(P[1][1], q, l[2], l[3]);
                if (KIND == kScanHgrn2) {
                    load_frag_a(ql, ops + kChunkT * kPitch + ks * 16, kPitch);
                    mma_16816(P[2][0], ql, h[0], h[1]), mma_16816(P[2][1], ql, h[2], h[3]);
                }
            }
#pragma unroll
            for (int i = 0; i < 2; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) O[i][e] += P[0][i][e] + (P[1][i][e] + P[2][i][e]);
            // the sums inside the chunk
            float A[8];  // A rows t = g, g + 8 at s = 2c, 2c + 1 | 2c + 8, 2c + 9, in operand order
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                const int t = g + ((e >> 1) & 1) * 8, s = 2 * c + (e & 1) + (e >> 2) * 8;
                A[e] = s <= t ? mat[t * 16 + s] : 0.0f;
                if (KIND == kScanMamba2 && s <= t) A[e] *= expf(tail[16 + t] - tail[16 + s]) * tail[s];
            }
            if (KIND == kScanMamba2) {
                const float e0 = expf(tail[16 + g]), e1 = expf(tail[16 + g + 8]);
#pragma unroll
                for (int i = 0; i < 2; ++i) O[i][0] *= e0, O[i][1] *= e0, O[i][2] *= e1, O[i][3] *= e1;
            }
            uint32_t ah[4], al[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) split_bf16(A[2 * e], A[2 * e + 1], &ah[e], &al[e]);
            mma_16816(O[0], ah, xv[0], xv[1]), mma_16816(O[1], ah, xv[2], xv[3]);
            mma_16816(O[0], al, xv[0], xv[1]), mma_16816(O[1], al, xv[2], xv[3]);
            const float skip = KIND == kScanMamba2 ? a.d_skip[head] : 0.0f;
#pragma unroll
            for (int i = 0; i < 2; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int tl = g + (e >> 1) * 8, t = chunk * kChunkT + tl, vl = warp * 16 + i * 8 + 2 * c + (e & 1);
                    if (t >= a.tokens || v0 + vl >= a.vdim) continue;
                    float y = O[i][e];
                    if (KIND == kScanMamba2) y += skip * __bfloat162float(xs[tl * kVPitch + vl]);
                    a.y[size_t(t) * inner + head * a.vdim + v0 + vl] = y;
                }
            // the state after the chunk
            if (KIND == kScanMamba2) {
                const float total = tail[16 + 15], decay = expf(total);
                uint32_t xh[4], xl[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) {  // operand e: columns of x in registers {0, 2, 1, 3}, tokens 2c, 2c + 1 (e < 2) or 2c + 8, 2c + 9
                    const uint32_t r = xv[((e & 1) << 1) | (e >> 1)];
                    const int s = 2 * c + (e >> 1) * 8;
                    split_bf16(__uint_as_float(r << 16) * (tail[s] * expf(total - tail[16 + s])), __uint_as_float(r & 0xffff0000u) * (tail[s + 1] * expf(total - tail[16 + s + 1])), &xh[e], &xl[e]);
                }
#pragma unroll
                for (int j = 0; j < ROWS / 8; j += 2) {
                    uint32_t k[4];
                    load_frag_b(k, ops + kChunkT * kPitch + j * 8, kPitch);
#pragma unroll
                    for (int h = 0; h < 2; ++h) {
#pragma unroll
                        for (int e = 0; e < 4; ++e) S[j + h][e] *= decay;
                        mma_16816(S[j + h], xh, k[2 * h], k[2 * h + 1]);
                        mma_16816(S[j + h], xl, k[2 * h], k[2 * h + 1]);
                    }
                }
            } else {
                const uint32_t xt[4] = {xv[0], xv[2], xv[1], xv[3]};
#pragma unroll
                for (int j = 0; j < ROWS / 8; j += 2) {
                    uint32_t kh[4], kl[4];
                    load_frag_b(kh, ops + 2 * kChunkT * kPitch + j * 8, kPitch);
                    load_frag_b(kl, ops + 3 * kChunkT * kPitch + j * 8, kPitch);
#pragma unroll
                    for (int h = 0; h < 2; ++h) {
                        const float2 fe = *reinterpret_cast<const float2*>(tail + (j + h) * 8 + 2 * c);
                        S[j + h][0] *= fe.x, S[j + h][1] *= fe.y, S[j + h][2] *= fe.x, S[j + h][3] *= fe.y;
                        mma_16816(S[j + h], xt, kh[2 * h], kh[2 * h + 1]);
                        mma_16816(S[j + h], xt, kl[2 * h], kl[2 * h + 1]);
                    }
                }
            }
        }
    }
#pragma unroll
    for (int j = 0; j < ROWS / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int v = vw + g + (e >> 1) * 8, d = 8 * j + 2 * c + (e & 1);
            if (v < a.vdim && d < a.n) state[size_t(v) * a.n + d] = S[j][e];
        }
}

}  // namespace qtb
