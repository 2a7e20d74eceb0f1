// Gated linear recurrences, one state matrix per head:
//
//   S_t = a_t (.) S_(t-1) + k_t x_t^T      y_t = S_t^T q_t       (S: N rows x vdim columns; a_t: a number or one per row)
//
// Three ways to make a, k, q and x from a layer's projections (ScanKind):
//   mamba2  a = exp(-exp(A_log) dt), k = dt B, q = C, with dt = softplus(dt_raw + dt_bias); x, B and C come out of a causal convolution
//           per channel and silu; the result is y + D x, times silu(z)
//   retention  a: a constant per head, q and k rotated by their position, k times N^(-1/2), x = v
//   hgrn2   a = l + (1 - l) sigmoid(f_raw + f_bias), k = 1 - a, q = silu(q_raw), x = v
// All of it in 32-bit arithmetic. The output norm follows in the kernel that consumes y (dense_gemv.cuh).
//
// A sequence's state lies in device memory as [head][vdim][N] floats and, for the convolution, a ring of its last `taps` raw inputs
// [tap slot][channel], position p in slot p % taps. Both belong to a slot of the sequence store. At position 0 the state counts as zero and
// inputs before the start as zero, so a slot needs no clearing when it is used again.
#pragma once
#include "dense_gemv.cuh"
#include "rotation.cuh"

namespace qtb {

enum ScanKind : int { kScanMamba2 = 0, kScanHgrn2 = 1, kScanRetention = 2 };

struct ScanArgs {
    int tokens;               // consecutive tokens of a sequence in this launch (1: a decode step, sequences in gridDim.z)
    const uint32_t* pos;      // positions as SeqIndex describes them
    SeqIndex seq;
    const float* p;           // projections [token][ld]; mamba2: z | x | B | C | dt, hgrn2: q | f | v, retention: q | k | v | g
    int ld;
    int heads, vdim, n;       // n: rows of the state
    int groups;               // mamba2: B and C are shared by heads / groups heads
    int taps;
    const float *conv_w, *conv_b, *dt_bias, *a_log, *d_skip;  // mamba2
    const float *f_bias, *lower;                              // hgrn2, heads * n each
    const float* decay;       // retention, one per head
    const double* turns;      // retention: turns of a rotated pair per position, rot_dims / 2 of them (rotation.cuh)
    int rot_dims;
    float* state;             // [slot][heads][vdim][n]
    float* conv;              // [slot][taps][conv channels]
    float* y;                 // [token][heads * vdim]
};

__device__ __forceinline__ float softplus_f(float v) { return v > 20.0f ? v + log1pf(expf(-v)) : log1pf(expf(v)); }

// Channel c of the convolution (x | B | C) at token t of the launch (position pos), with silu. row: the token's row of the projections.
__device__ __forceinline__ float conv_silu(const ScanArgs& a, const float* ring, int row, int t, uint32_t pos, int c, int channels, int inner) {
    float s = a.conv_b[c];
    const float* w = a.conv_w + size_t(c) * a.taps;
    for (int k0 = 0; k0 < a.taps; k0 += 4) {
        float v[4], f[4];  // four taps' loads in flight
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const int back = a.taps - 1 - k0 - k;
            const bool there = back >= 0 && static_cast<uint32_t>(back) <= pos;  // not before the start of the sequence
            const float* src = back <= t ? a.p + size_t(row - back) * a.ld + inner + c : ring + size_t((pos - back) % a.taps) * channels + c;
            v[k] = there ? *src : 0.0f, f[k] = there ? w[k0 + k] : 0.0f;
        }
#pragma unroll
        for (int k = 0; k < 4; ++k) s = fmaf(f[k], v[k], s);
    }
    return silu_f(s);
}

constexpr int kScanThreads = 128, kScanRows = 16;  // columns of S (values) per block: four per warp
constexpr int kScanStage = 16;                     // tokens whose a, k, q, x are staged at a time
constexpr int kScanMaxPer = 8;                     // rows of S per lane: n <= 256

inline size_t scan_smem(int n) { return (size_t(kScanStage) * (3 * n + kScanRows) + 2 * kScanStage) * sizeof(float); }

// grid: (heads, ceil(vdim / kScanRows), sequences). A warp keeps four columns of S in registers, the rows spread over its lanes.
template <int KIND>
__global__ void __launch_bounds__(kScanThreads) gated_scan_kernel(const __grid_constant__ ScanArgs a) {
    extern __shared__ float scan_sm[];
    pdl_trigger();
    const int n = a.n, head = blockIdx.x, v0 = blockIdx.y * kScanRows, z = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    float *ks = scan_sm, *qs = ks + kScanStage * n, *as = qs + kScanStage * n, *xs = as + kScanStage * n, *one = xs + kScanStage * kScanRows;
    const uint32_t slot = a.seq.pos_stride != 0 ? seq_of(a.seq, z) : 0, pos0 = seq_position(a.seq, a.pos, z);
    const int inner = a.heads * a.vdim, channels = inner + 2 * a.groups * n, row0 = z * a.tokens;
    const float* ring = KIND == kScanMamba2 ? a.conv + size_t(slot) * a.taps * channels : nullptr;
    const int group = KIND == kScanMamba2 ? head / (a.heads / a.groups) : 0;
    float* state = a.state + ((size_t(slot) * a.heads + head) * a.vdim) * n;
    const int mine = v0 + warp * 4;  // first of this warp's four columns
    float s[4][kScanMaxPer];
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int e = 0; e < kScanMaxPer; ++e) {
            const int i = lane + 32 * e;
            s[j][e] = pos0 > 0 && mine + j < a.vdim && i < n ? state[size_t(mine + j) * n + i] : 0.0f;
        }
    pdl_wait();  // (the state above was written by an earlier step)
    for (int t0 = 0; t0 < a.tokens; t0 += kScanStage) {
        const int nt = min(kScanStage, a.tokens - t0);
        __syncthreads();
        if (KIND == kScanMamba2) {
            for (int i = tid; i < nt; i += kScanThreads) {
                const float dt = softplus_f(a.p[size_t(row0 + t0 + i) * a.ld + inner + channels + head] + a.dt_bias[head]);
                one[i] = dt, one[kScanStage + i] = expf(-expf(a.a_log[head]) * dt);
            }
            for (int i = tid; i < nt * n; i += kScanThreads) {
                const int t = i / n, c = i % n;
                ks[i] = conv_silu(a, ring, row0 + t0 + t, t0 + t, pos0 + t0 + t, inner + group * n + c, channels, inner);
                qs[i] = conv_silu(a, ring, row0 + t0 + t, t0 + t, pos0 + t0 + t, inner + a.groups * n + group * n + c, channels, inner);
            }
            for (int i = tid; i < nt * kScanRows; i += kScanThreads) {
                const int t = i / kScanRows, v = v0 + i % kScanRows;
                xs[i] = v < a.vdim ? conv_silu(a, ring, row0 + t0 + t, t0 + t, pos0 + t0 + t, head * a.vdim + v, channels, inner) : 0.0f;
            }
        } else if (KIND == kScanRetention) {
            const float scale = 1.0f / sqrtf(static_cast<float>(n));
            const int half = a.rot_dims / 2, items = n - half;  // an item is a rotated pair, or an element that stays as it is
            for (int i = tid; i < nt * items; i += kScanThreads) {
                const int t = i / items, j = i % items;
                const float* p = a.p + size_t(row0 + t0 + t) * a.ld + head * n;
                const float* pk = p + a.heads * n;
                if (j < half) {
                    const float2 cs = rotation(a.turns[j], pos0 + t0 + t);
                    const float2 q = rotate_pair(p[j], p[j + half], cs), k = rotate_pair(pk[j], pk[j + half], cs);
                    qs[t * n + j] = q.x, qs[t * n + j + half] = q.y;
                    ks[t * n + j] = k.x * scale, ks[t * n + j + half] = k.y * scale;
                } else {
                    qs[t * n + j + half] = p[j + half], ks[t * n + j + half] = pk[j + half] * scale;
                }
            }
            for (int i = tid; i < nt * kScanRows; i += kScanThreads) {
                const int t = i / kScanRows, v = v0 + i % kScanRows;
                xs[i] = v < a.vdim ? a.p[size_t(row0 + t0 + t) * a.ld + 2 * a.heads * n + head * a.vdim + v] : 0.0f;
            }
        } else {
            for (int i = tid; i < nt * n; i += kScanThreads) {
                const int t = i / n, c = head * n + i % n;
                const float* p = a.p + size_t(row0 + t0 + t) * a.ld;
                const float f = p[a.heads * n + c] + a.f_bias[c], l = a.lower[c];
                qs[i] = silu_f(p[c]);
                as[i] = l + (1.0f - l) * sigmoid_f(f);
                ks[i] = (1.0f - l) * sigmoid_f(-f);
            }
            for (int i = tid; i < nt * kScanRows; i += kScanThreads) {
                const int t = i / kScanRows, v = v0 + i % kScanRows;
                xs[i] = v < a.vdim ? a.p[size_t(row0 + t0 + t) * a.ld + 2 * a.heads * n + head * a.vdim + v] : 0.0f;
            }
        }
        __syncthreads();
        for (int t = 0; t < nt; ++t) {
            float x[4], acc[4] = {};
#pragma unroll
            for (int j = 0; j < 4; ++j) x[j] = xs[t * kScanRows + warp * 4 + j];
            const float decay = KIND == kScanMamba2 ? one[kScanStage + t] : KIND == kScanRetention ? a.decay[head] : 0.0f, step = KIND == kScanMamba2 ? one[t] : 1.0f;
#pragma unroll
            for (int e = 0; e < kScanMaxPer; ++e) {
                const int i = lane + 32 * e;
                if (i < n) {
                    const float k = ks[t * n + i] * step, q = qs[t * n + i], d = KIND != kScanHgrn2 ? decay : as[t * n + i];
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        s[j][e] = d * s[j][e] + k * x[j];
                        acc[j] = fmaf(s[j][e], q, acc[j]);
                    }
                }
            }
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                acc[j] = warp_sum(acc[j]);
                const int v = mine + j;
                if (lane == j && v < a.vdim) {
                    const size_t row = row0 + t0 + t;
                    float y = acc[j];
                    if (KIND == kScanMamba2) y = (y + a.d_skip[head] * x[j]) * silu_f(a.p[row * a.ld + head * a.vdim + v]);
                    a.y[row * inner + head * a.vdim + v] = y;
                }
            }
        }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int e = 0; e < kScanMaxPer; ++e) {
            const int i = lane + 32 * e;
            if (mine + j < a.vdim && i < n) state[size_t(mine + j) * n + i] = s[j][e];
        }
    // The raw inputs of the convolution: a single token writes its own slot, which no block of this launch reads. Longer launches leave
    // this to conv_tail_kernel, because their last tokens fall into slots that other blocks may still have to read.
    if (KIND == kScanMamba2 && a.tokens == 1) {
        float* mine_ring = a.conv + size_t(slot) * a.taps * channels + size_t(pos0 % a.taps) * channels;
        const float* raw = a.p + size_t(row0) * a.ld + inner;
        for (int i = tid; i < kScanRows; i += kScanThreads)
            if (v0 + i < a.vdim) mine_ring[head * a.vdim + v0 + i] = raw[head * a.vdim + v0 + i];
        if (blockIdx.y == 0 && head % (a.heads / a.groups) == 0)
            for (int i = tid; i < n; i += kScanThreads) {
                mine_ring[inner + group * n + i] = raw[inner + group * n + i];
                mine_ring[inner + (a.groups + group) * n + i] = raw[inner + (a.groups + group) * n + i];
            }
    }
}

// After a launch of several tokens: the last `taps` raw inputs of every channel go to the ring. grid: (channels / 256)
__global__ void conv_tail_kernel(const __grid_constant__ ScanArgs a) {
    const int inner = a.heads * a.vdim, channels = inner + 2 * a.groups * a.n, c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= channels) return;
    const uint32_t slot = a.seq.pos_stride != 0 ? seq_of(a.seq, 0) : 0, pos0 = seq_position(a.seq, a.pos, 0);
    float* ring = a.conv + size_t(slot) * a.taps * channels;
    for (int t = max(0, a.tokens - a.taps); t < a.tokens; ++t) ring[size_t((pos0 + t) % a.taps) * channels + c] = a.p[size_t(t) * a.ld + inner + c];
}

}  // namespace qtb
