// Dense (16- or 32-bit) projections of one token, fused with what stands before and after them: the kernels a layered decoder
// (layered.cuh) takes a decode step with. Activations and sums are 32-bit; an activation is rounded to the storage type where the
// batched path (dense_gemm_tc.cuh) stores it, so both paths round in the same places.
//
//   norm_project_kernel    norms of the residual stream (to which the normed results of two mixers may still have to be added), then up to
//                          two stacked projections of them, each row range with its own ending (plain, sigmoid of a gate, SwiGLU of
//                          interleaved gate | up rows)
//   finish_project_kernel  the mixer's output norm, then output and down projection, both gates and the residual sum
//   out_project_kernel     output norm and gate of one mixer or two side by side, then their output projections
//
// The kernels of a decode step follow one another with programmatic dependent launch: a kernel may start while the one before it still runs,
// brings what does not depend on it (weights, states, cached keys) on the way, and only then waits for its results.
//
// A warp owns two rows (one in the second kernel) and streams them with 16-byte loads, four per row in flight and lane; the activation
// vector lies in shared memory as floats.
#pragma once
#include <cstdint>
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "decode.cuh"

namespace qtb {

typedef __nv_bfloat16 bf16;

constexpr int kRowPad = 128;   // a stacked projection's row ranges start at multiples of this (the M of a tensor-core tile)
constexpr int kColPad = 64;    // columns are padded with zeros to a multiple of this (a 128-byte swizzled TMA box)

template <typename T> __device__ __forceinline__ T to_storage(float v);
template <> __device__ __forceinline__ float to_storage<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 to_storage<bf16>(float v) { return __float2bfloat16_rn(v); }
__device__ __forceinline__ float from_storage(float v) { return v; }
__device__ __forceinline__ float from_storage(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ float round_to(float v) { return from_storage(to_storage<T>(v)); }
__device__ __forceinline__ float sigmoid_f(float v) { return 1.0f / (1.0f + expf(-v)); }
__device__ __forceinline__ float silu_f(float v) { return v / (1.0f + expf(-v)); }

// Programmatic dependent launch: the next kernel of the stream may start / everything the kernels before this one wrote is visible. Both do
// nothing in a kernel that was launched without the attribute.
__device__ __forceinline__ void pdl_trigger() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
template <typename... P, typename... A>
inline cudaError_t launch_dependent(void (*kernel)(P...), dim3 grid, int threads, size_t smem, cudaStream_t s, const A&... args) {
    cudaLaunchConfig_t cfg{};
    cudaLaunchAttribute attr{};
    attr.id = cudaLaunchAttributeProgrammaticStreamSerialization, attr.val.programmaticStreamSerializationAllowed = 1;
    cfg.gridDim = grid, cfg.blockDim = dim3(threads), cfg.dynamicSmemBytes = smem, cfg.stream = s, cfg.attrs = &attr, cfg.numAttrs = 1;
    return cudaLaunchKernelEx(&cfg, kernel, static_cast<P>(args)...);
}
// `bytes` (a multiple of 16) from p on are requested into L2.
__device__ __forceinline__ void l2_prefetch(const void* p, size_t bytes) {
    asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(p), "r"(static_cast<uint32_t>(bytes)) : "memory");
}

// What becomes of the rows of one range of a stacked projection.
enum SegKind : int { kSegPlain = 0, kSegSigmoid = 1, kSegSwiGlu = 2, kSegStore = 3 };
struct DenseSeg {
    int row0, rows;      // rows of the stack (row0 a multiple of kRowPad)
    int kind;
    int ld;              // elements between the results of consecutive tokens
    float* f;            // kSegPlain, kSegSigmoid: 32-bit results
    void* t;             // kSegSwiGlu: silu(row 2 i) * row 2 i + 1, in the storage type; kSegStore: results in the storage type
    const float* bias;   // kSegSigmoid: added before the sigmoid, may be nullptr
};
struct DenseStack {
    const void* w;       // [rows padded][pitch], storage type
    int pitch, cols;     // pitch: columns padded to kColPad
    int n_seg;
    DenseSeg seg[4];
};
// The range that row `row` of a stack belongs to.
__device__ __forceinline__ const DenseSeg& dense_seg_of(const DenseStack& st, int row) {
    int k = 0;
    while (k + 1 < st.n_seg && row >= st.seg[k + 1].row0) ++k;
    return st.seg[k];
}

// A norm over the model width: RMS (x / rms(x)) w, or, element by element, tanh(alpha x) w + b.
struct NormParams {
    const float* w;
    const float* b;      // not nullptr: the tanh form
    float alpha;
};
__device__ __forceinline__ float norm_value(const NormParams& n, float x, float inv, int i) {
    return n.b != nullptr ? tanhf(n.alpha * x) * __ldg(n.w + i) + __ldg(n.b + i) : x * inv * __ldg(n.w + i);
}

// Two vectors whose RMS norms, each with its weight, are averaged and added to the residual stream.
struct PairSum {
    const float* r[2];   // [tokens][width]; nullptr: nothing is added
    const float* w[2];
};

// ---- reductions ---------------------------------------------------------------------------------------------------------------------
__device__ __forceinline__ float warp_sum(float v) {
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float2 block_sum2(float2 v, float2* sh) {  // two sums at once; sh: one float2 per warp
    v = make_float2(warp_sum(v.x), warp_sum(v.y));
    const int w = threadIdx.x >> 5, nw = blockDim.x >> 5;
    __syncthreads();
    if ((threadIdx.x & 31) == 0) sh[w] = v;
    __syncthreads();
    float2 t = make_float2(0.0f, 0.0f);
    for (int i = 0; i < nw; ++i) t.x += sh[i].x, t.y += sh[i].y;
    return t;
}
__device__ __forceinline__ float block_sum(float v, float* sh) {  // sh: one float per warp
    v = warp_sum(v);
    const int w = threadIdx.x >> 5, nw = blockDim.x >> 5;
    __syncthreads();
    if ((threadIdx.x & 31) == 0) sh[w] = v;
    __syncthreads();
    float t = 0.0f;
    for (int i = 0; i < nw; ++i) t += sh[i];
    return t;
}

// ---- activation vector in shared memory ----------------------------------------------------------------------------------------------
// 16-bit weights: a lane multiplies eight columns per load; the two halves of an eight lie in two separate arrays so that its 16-byte
// reads fall on different banks. 32-bit weights: four columns per load, plain order.
template <typename T> __device__ __forceinline__ int act_index(int e, int pitch);
template <> __device__ __forceinline__ int act_index<float>(int e, int) { return e; }
template <> __device__ __forceinline__ int act_index<bf16>(int e, int pitch) { return ((e >> 2) & 1) * (pitch >> 1) + ((e >> 3) << 2) + (e & 3); }

__device__ __forceinline__ uint4 load_stream(const void* p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}
__device__ __forceinline__ float dot_piece(const uint4& w, const float* h, int piece, int pitch, bf16) {
    const float4 a = *reinterpret_cast<const float4*>(h + piece * 4), b = *reinterpret_cast<const float4*>(h + (pitch >> 1) + piece * 4);
    float s = __uint_as_float(w.x << 16) * a.x;
    s = fmaf(__uint_as_float(w.x & 0xffff0000u), a.y, s);
    s = fmaf(__uint_as_float(w.y << 16), a.z, s);
    s = fmaf(__uint_as_float(w.y & 0xffff0000u), a.w, s);
    s = fmaf(__uint_as_float(w.z << 16), b.x, s);
    s = fmaf(__uint_as_float(w.z & 0xffff0000u), b.y, s);
    s = fmaf(__uint_as_float(w.w << 16), b.z, s);
    return fmaf(__uint_as_float(w.w & 0xffff0000u), b.w, s);
}
__device__ __forceinline__ float dot_piece(const uint4& w, const float* h, int piece, int, float) {
    const float4 a = *reinterpret_cast<const float4*>(h + piece * 4);
    float s = __uint_as_float(w.x) * a.x;
    s = fmaf(__uint_as_float(w.y), a.y, s);
    s = fmaf(__uint_as_float(w.z), a.z, s);
    return fmaf(__uint_as_float(w.w), a.w, s);
}

// Four consecutive elements (e a multiple of 4) of an activation vector, and eight of the storage type.
template <typename T> __device__ __forceinline__ void act_put4(float* h, int e, int pitch, float4 v) { *reinterpret_cast<float4*>(h + act_index<T>(e, pitch)) = v; }
__device__ __forceinline__ void act_put_storage(float* h, int piece, int pitch, const bf16* src) {
    const uint4 w = *reinterpret_cast<const uint4*>(src + piece * 8);
    const auto lo = [](uint32_t u) { return __uint_as_float(u << 16); };
    const auto hi = [](uint32_t u) { return __uint_as_float(u & 0xffff0000u); };
    act_put4<bf16>(h, piece * 8, pitch, make_float4(lo(w.x), hi(w.x), lo(w.y), hi(w.y)));
    act_put4<bf16>(h, piece * 8 + 4, pitch, make_float4(lo(w.z), hi(w.z), lo(w.w), hi(w.w)));
}
__device__ __forceinline__ void act_put_storage(float* h, int piece, int, const float* src) {
    *reinterpret_cast<float4*>(h + piece * 4) = *reinterpret_cast<const float4*>(src + piece * 4);
}

// The first pieces of R consecutive rows, in registers: they can be on their way before the vector is known.
template <int R> struct RowHead { uint4 v[R][8 / R]; };
template <typename T, int R>
__device__ __forceinline__ void load_pieces(RowHead<R>& b, const T* w, int pitch, int p0) {
    constexpr int kPer = 16 / sizeof(T);
    const int pieces = pitch / kPer;
#pragma unroll
    for (int u = 0; u < 8 / R; ++u)
#pragma unroll
        for (int r = 0; r < R; ++r) b.v[r][u] = p0 + 32 * u < pieces ? load_stream(w + size_t(r) * pitch + size_t(p0 + 32 * u) * kPer) : make_uint4(0, 0, 0, 0);
}
// Sums of R consecutive rows over the vector h (shared memory), the rows' first pieces in `head`: every lane returns the whole sums.
template <typename T, int R>
__device__ __forceinline__ void dot_rows(const T* w, int pitch, const float* h, RowHead<R>& head, float (&sum)[R]) {
    constexpr int kPer = 16 / sizeof(T), U = 8 / R;
    const int pieces = pitch / kPer, lane = threadIdx.x & 31;
#pragma unroll
    for (int r = 0; r < R; ++r) sum[r] = 0.0f;
    for (int p0 = lane; p0 < pieces; p0 += 32 * U) {
        if (p0 != lane) load_pieces<T, R>(head, w, pitch, p0);
#pragma unroll
        for (int u = 0; u < U; ++u)
            if (p0 + 32 * u < pieces) {
#pragma unroll
                for (int r = 0; r < R; ++r) sum[r] += dot_piece(head.v[r][u], h, p0 + 32 * u, pitch, T());
            }
    }
#pragma unroll
    for (int r = 0; r < R; ++r) sum[r] = warp_sum(sum[r]);
}

// ---- norms and the projections of their results ----------------------------------------------------------------------------------------
struct NormProjectArgs {
    const float* x;             // residual stream, [tokens][width]
    NormParams norm[2];
    float eps;
    int width, n_stack;         // projections: 1 or 2, each over its own norm of x
    DenseStack stack[2];
    PairSum pair;               // added to x first; the first block writes the sum to x_out (not x itself)
    float* x_out;
    void* h_out;                // the first norm's result in the storage type, [tokens][pitch]; may be nullptr
};

constexpr int kProjectThreads = 256;

// FORM: what stands before the projections is known when the kernel is compiled, which keeps it short. kProjectRms: RMS norms; kProjectTanh: the tanh
// norm; kProjectAny: either, of a pair sum (both of the latter also write h_out).
enum ProjectForm : int { kProjectRms = 0, kProjectTanh = 1, kProjectAny = 2 };
template <typename T, int FORM>
__global__ void __launch_bounds__(kProjectThreads, 4) norm_project_kernel(NormProjectArgs a) {
    extern __shared__ float act_smem[];
    __shared__ float red[kProjectThreads / 32];
    __shared__ float2 red2[kProjectThreads / 32];
    const int tid = threadIdx.x, token = blockIdx.y, pitch = a.stack[0].pitch;
    const float* x = a.x + size_t(token) * a.width;
    const int warps = gridDim.x * (kProjectThreads / 32);
    int unit = blockIdx.x * (kProjectThreads / 32) + (tid >> 5);
    pdl_trigger();
    RowHead<2> head;  // the rows this warp begins with
    {
        int u = unit;
        for (int s = 0; s < a.n_stack; ++s)
            for (int k = 0; k < a.stack[s].n_seg; ++k) {
                const int units = (a.stack[s].seg[k].rows + 1) / 2;
                if (u >= 0 && u < units) load_pieces<T, 2>(head, static_cast<const T*>(a.stack[s].w) + size_t(a.stack[s].seg[k].row0 + 2 * u) * pitch, pitch, tid & 31);
                u -= units;
            }
    }
    bool first = true;
    if (FORM != kProjectRms && blockIdx.x == 0 && tid == 0 && a.width >= 4) {  // vectors that every block reads after the wait
        const uint32_t bytes = a.width * 4 & ~15;
        l2_prefetch(a.norm[0].w, bytes);
        if (a.norm[0].b != nullptr) l2_prefetch(a.norm[0].b, bytes);
        if (a.pair.r[0] != nullptr) l2_prefetch(a.pair.w[0], bytes), l2_prefetch(a.pair.w[1], bytes);
    }
    pdl_wait();
    if (FORM == kProjectAny && a.pair.r[0] != nullptr) {
        float* sum = act_smem + a.n_stack * pitch;
        const float *l = a.pair.r[0] + size_t(token) * a.width, *r = a.pair.r[1] + size_t(token) * a.width;
        float sl = 0.0f, sr = 0.0f;
#pragma unroll 4
        for (int i = tid; i < a.width; i += kProjectThreads) sl += l[i] * l[i], sr += r[i] * r[i];
        const float2 both = block_sum2(make_float2(sl, sr), red2);
        sl = both.x, sr = both.y;
        const float il = 0.5f / sqrtf(sl / static_cast<float>(a.width) + a.eps), ir = 0.5f / sqrtf(sr / static_cast<float>(a.width) + a.eps);
#pragma unroll 4
        for (int i = tid; i < a.width; i += kProjectThreads) {
            const float v = x[i] + (l[i] * il * a.pair.w[0][i] + r[i] * ir * a.pair.w[1][i]);
            sum[i] = v;
            if (blockIdx.x == 0) a.x_out[size_t(token) * a.width + i] = v;
        }
        x = sum;  // (each thread reads back what it wrote)
    }
    float inv = 1.0f;
    if (FORM == kProjectRms || (FORM == kProjectAny && a.norm[0].b == nullptr)) {
        float ss = 0.0f;
#pragma unroll 4
        for (int i = tid; i < a.width; i += kProjectThreads) ss += x[i] * x[i];
        inv = 1.0f / sqrtf(block_sum(ss, red) / static_cast<float>(a.width) + a.eps);
    }
    for (int s = 0; s < a.n_stack; ++s)
#pragma unroll 4
        for (int i = tid; i < pitch; i += kProjectThreads) {
            const float v = i < a.width ? round_to<T>(FORM == kProjectRms    ? x[i] * inv * a.norm[s].w[i]
                                                        : FORM == kProjectTanh ? tanhf(a.norm[s].alpha * x[i]) * a.norm[s].w[i] + a.norm[s].b[i]
                                                                               : norm_value(a.norm[s], x[i], inv, i))
                                          : 0.0f;
            act_smem[s * pitch + act_index<T>(i, pitch)] = v;
            if (FORM != kProjectRms && a.h_out != nullptr && s == 0 && blockIdx.x == 0) static_cast<T*>(a.h_out)[size_t(token) * pitch + i] = to_storage<T>(v);
        }
    __syncthreads();
    for (int s = 0; s < a.n_stack; ++s)
        for (int k = 0; k < a.stack[s].n_seg; ++k) {
            const DenseSeg& g = a.stack[s].seg[k];
            const int units = (g.rows + 1) / 2;
            for (; unit < units; unit += warps) {
                const int r = unit * 2;
                float v[2];  // (an odd last row has a row of padding behind it: row ranges are padded to kRowPad)
                const T* rows = static_cast<const T*>(a.stack[s].w) + size_t(g.row0 + r) * pitch;
                if (!first) load_pieces<T, 2>(head, rows, pitch, tid & 31);
                first = false;
                dot_rows<T, 2>(rows, pitch, act_smem + s * pitch, head, v);
                if ((tid & 31) != 0) continue;
                if (g.kind == kSegSwiGlu) {
                    static_cast<T*>(g.t)[size_t(token) * g.ld + unit] = to_storage<T>(silu_f(v[0]) * v[1]);
                } else {
                    float* f = g.f + size_t(token) * g.ld + r;
                    for (int j = 0; j < 2 && r + j < g.rows; ++j) f[j] = g.kind == kSegSigmoid ? sigmoid_f(v[j] + (g.bias != nullptr ? g.bias[r + j] : 0.0f)) : v[j];
                }
            }
            unit -= units;
        }
}

// ---- output norm of a mixer -----------------------------------------------------------------------------------------------------------
// y of one token in `parts` equal parts, each divided by its own root mean square, times w[i % w_len], or with GATED times silu(gate[i]) instead
// (gate may be nullptr); in place in shared memory, in the order act_index<T>. red: one float per warp.
template <typename T, bool GATED>
__device__ __forceinline__ void parts_norm(float* y, int n, int pitch, int parts, float eps, const float* w, int w_len, const float* gate, float* red) {
    const auto ending = [&](float v, int e) {
        if constexpr (GATED) return round_to<T>(gate != nullptr ? v * silu_f(gate[e]) : v);
        else return round_to<T>(v * w[e % w_len]);
    };
    const int len = n / parts, warps = blockDim.x >> 5, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (parts >= warps) {  // a warp per part
        for (int p = warp; p < parts; p += warps) {
            float ss = 0.0f;
            for (int i = lane; i < len; i += 32) {
                const float v = y[act_index<T>(p * len + i, pitch)];
                ss += v * v;
            }
            const float inv = 1.0f / sqrtf(warp_sum(ss) / static_cast<float>(len) + eps);
            for (int i = lane; i < len; i += 32) {
                const int e = p * len + i, at = act_index<T>(e, pitch);
                y[at] = ending(y[at] * inv, e);
            }
        }
        __syncthreads();
        return;
    }
    for (int p = 0; p < parts; ++p) {
        float ss = 0.0f;
        for (int i = threadIdx.x; i < len; i += blockDim.x) {
            const float v = y[act_index<T>(p * len + i, pitch)];
            ss += v * v;
        }
        const float inv = 1.0f / sqrtf(block_sum(ss, red) / static_cast<float>(len) + eps);
        for (int i = threadIdx.x; i < len; i += blockDim.x) {
            const int e = p * len + i, at = act_index<T>(e, pitch);
            y[at] = ending(y[at] * inv, e);
        }
    }
    __syncthreads();
}

// ---- output and down projection, gates, residual ------------------------------------------------------------------------------------------
struct FinishProjectArgs {
    float* x;                   // residual stream, updated in place: x += (W_o y) * gate1 + (W_down m) * gate2
    int width;
    const float* y;             // the mixer's output, 32-bit; normed here when norm_parts > 0
    int inner;
    int norm_parts, norm_len;   // norm_len: length of the weight vector (inner, or a head's vdim)
    const float* norm_w;
    float eps;
    const void* o;              // [width][o_pitch]
    int o_pitch;
    const void* m;              // feed-forward activations in the storage type, [tokens][down_pitch]; nullptr: no feed-forward
    const void* down;           // [width][down_pitch]
    int down_pitch;
    const float *gate1, *gate2; // sigmoids, [tokens][width]; nullptr: no gate
};

template <typename T>
__global__ void __launch_bounds__(kProjectThreads, 4) finish_project_kernel(FinishProjectArgs a) {
    extern __shared__ float act_smem[];
    __shared__ float red[kProjectThreads / 32];
    const int tid = threadIdx.x, lane = tid & 31, token = blockIdx.y;
    float *y = act_smem, *m = act_smem + a.o_pitch;
    const int warps = gridDim.x * (kProjectThreads / 32);
    pdl_trigger();
    RowHead<1> head;
    bool first = true;
    if (const int row = blockIdx.x * (kProjectThreads / 32) + (tid >> 5); row < a.width) {
        load_pieces<T, 1>(head, static_cast<const T*>(a.o) + size_t(row) * a.o_pitch, a.o_pitch, lane);
        if (lane == 0) {
            l2_prefetch(static_cast<const T*>(a.o) + size_t(row) * a.o_pitch, a.o_pitch * sizeof(T));
            if (a.m != nullptr) l2_prefetch(static_cast<const T*>(a.down) + size_t(row) * a.down_pitch, a.down_pitch * sizeof(T));
        }
    }
    pdl_wait();
    const float* yt = a.y + size_t(token) * a.inner;
    const bool norm = a.norm_parts > 0;
    if (a.inner % 4 == 0) {
#pragma unroll 4
        for (int i = tid * 4; i < a.o_pitch; i += kProjectThreads * 4) {
            float4 v = i < a.inner ? *reinterpret_cast<const float4*>(yt + i) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (!norm) v = make_float4(round_to<T>(v.x), round_to<T>(v.y), round_to<T>(v.z), round_to<T>(v.w));
            act_put4<T>(y, i, a.o_pitch, v);
        }
    } else {
        for (int i = tid; i < a.o_pitch; i += kProjectThreads) {
            const float v = i < a.inner ? yt[i] : 0.0f;
            y[act_index<T>(i, a.o_pitch)] = norm ? v : round_to<T>(v);
        }
    }
    if (a.m != nullptr) {
        constexpr int kPer = 16 / sizeof(T);
#pragma unroll 4
        for (int i = tid; i < a.down_pitch / kPer; i += kProjectThreads) act_put_storage(m, i, a.down_pitch, static_cast<const T*>(a.m) + size_t(token) * a.down_pitch);
    }
    __syncthreads();
    if (norm) parts_norm<T, false>(y, a.inner, a.o_pitch, a.norm_parts, a.eps, a.norm_w, a.norm_len, nullptr, red);
    for (int row = blockIdx.x * (kProjectThreads / 32) + (tid >> 5); row < a.width; row += warps) {
        float so[1], sd[1] = {0.0f};
        const T *o_row = static_cast<const T*>(a.o) + size_t(row) * a.o_pitch, *d_row = static_cast<const T*>(a.down) + size_t(row) * a.down_pitch;
        if (!first) load_pieces<T, 1>(head, o_row, a.o_pitch, lane);
        first = false;
        dot_rows<T, 1>(o_row, a.o_pitch, y, head, so);
        if (a.m != nullptr) {
            load_pieces<T, 1>(head, d_row, a.down_pitch, lane);
            dot_rows<T, 1>(d_row, a.down_pitch, m, head, sd);
        }
        if (lane == 0) {
            const size_t at = size_t(token) * a.width + row;
            const float g1 = a.gate1 != nullptr ? a.gate1[at] : 1.0f, g2 = a.gate2 != nullptr ? a.gate2[at] : 1.0f;
            a.x[at] += so[0] * g1 + sd[0] * g2;
        }
    }
}

// ---- output projections of one mixer, or of two side by side ------------------------------------------------------------------------------
struct OutProjectArgs {
    int width, n;               // n: mixers
    float eps;
    struct Mixer {
        const float* y;         // 32-bit output of the mixer, [tokens][inner]
        int inner, parts;       // parts > 0: each divided by its root mean square
        const float* gate;      // times silu(gate[token * gate_ld + i]); may be nullptr
        int gate_ld;
        const void* w;          // [width][pitch]
        int pitch;
        float* out;             // [tokens][width]
        bool add;               // out += W y instead of out = W y
    } mix[2];
};

template <typename T>
__global__ void __launch_bounds__(kProjectThreads, 4) out_project_kernel(const __grid_constant__ OutProjectArgs a) {
    extern __shared__ float act_smem[];
    __shared__ float red[kProjectThreads / 32];
    const int tid = threadIdx.x, lane = tid & 31, token = blockIdx.y, warps = gridDim.x * (kProjectThreads / 32), units = a.n * a.width;
    const int unit0 = blockIdx.x * (kProjectThreads / 32) + (tid >> 5);
    pdl_trigger();
    RowHead<1> head;
    bool first = true;
    if (unit0 < units) {
        const OutProjectArgs::Mixer& m = a.mix[unit0 >= a.width ? 1 : 0];
        const T* w = static_cast<const T*>(m.w) + size_t(unit0 % a.width) * m.pitch;
        load_pieces<T, 1>(head, w, m.pitch, lane);
        if (lane == 0) l2_prefetch(w, m.pitch * sizeof(T));
    }
    pdl_wait();
    float* gates = act_smem + a.mix[0].pitch + (a.n > 1 ? a.mix[1].pitch : 0);
    for (int k = 0; k < a.n; ++k) {
        const OutProjectArgs::Mixer& m = a.mix[k];
        // a block all of whose rows belong to the other mixer leaves this one's vector out
        const int lo = blockIdx.x * (kProjectThreads / 32), hi = lo + kProjectThreads / 32 - 1;
        if (warps >= units && (k == 0 ? lo >= a.width : hi < a.width)) continue;
        float* y = act_smem + (k > 0 ? a.mix[0].pitch : 0);
        const float *src = m.y + size_t(token) * m.inner, *gate = m.gate != nullptr ? m.gate + size_t(token) * m.gate_ld : nullptr;
#pragma unroll 8
        for (int i = tid; i < m.pitch; i += kProjectThreads) {
            const float v = i < m.inner ? src[i] : 0.0f, z = gate != nullptr && i < m.inner ? gate[i] : 0.0f;
            y[act_index<T>(i, m.pitch)] = m.parts > 0 ? v : round_to<T>(v);
            if (gate != nullptr && i < m.inner) gates[i] = z;
        }
        __syncthreads();
        if (m.parts > 0) parts_norm<T, true>(y, m.inner, m.pitch, m.parts, a.eps, nullptr, 1, gate != nullptr ? gates : nullptr, red);
        else __syncthreads();
    }
    for (int unit = unit0; unit < units; unit += warps) {
        const int k = unit >= a.width ? 1 : 0, row = unit - k * a.width;
        const OutProjectArgs::Mixer& m = a.mix[k];
        const T* w = static_cast<const T*>(m.w) + size_t(row) * m.pitch;
        float v[1];
        if (!first) load_pieces<T, 1>(head, w, m.pitch, lane);
        first = false;
        dot_rows<T, 1>(w, m.pitch, act_smem + (k > 0 ? a.mix[0].pitch : 0), head, v);
        if (lane == 0) {
            float* out = m.out + size_t(token) * a.width + row;
            *out = m.add ? *out + v[0] : v[0];
        }
    }
}

// ---- batched counterparts of the steps around the projections ------------------------------------------------------------------------------
// x = embed[token] * scale + pos[position] (pos may be nullptr)
template <typename T>
__global__ void embed_scaled_kernel(const T* embed, int pitch, const T* pos_table, const uint32_t* tokens, const uint32_t* pos, SeqIndex seq, float scale, int width, float* x) {
    const int i = blockIdx.x * blockDim.x + threadIdx.x, t = blockIdx.y;
    if (i >= width) return;
    float v = from_storage(embed[size_t(tokens[t]) * pitch + i]) * scale;
    if (pos_table != nullptr) v += from_storage(pos_table[size_t(seq_position(seq, pos, t)) * width + i]);
    x[size_t(t) * width + i] = v;
}

// h_s = norm s of x, in the storage type; rows (optional) picks tokens
template <typename T>
__global__ void __launch_bounds__(256) norm_rows_kernel(const float* x, int width, float eps, NormParams n0, T* h0, NormParams n1, T* h1, int pitch, const uint32_t* rows) {
    __shared__ float red[8];
    const int t = blockIdx.x;
    const float* xr = x + size_t(rows != nullptr ? rows[t] : t) * width;
    float inv = 1.0f;
    if (n0.b == nullptr) {
        float ss = 0.0f;
        for (int i = threadIdx.x; i < width; i += blockDim.x) ss += xr[i] * xr[i];
        inv = 1.0f / sqrtf(block_sum(ss, red) / static_cast<float>(width) + eps);
    }
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
        h0[size_t(t) * pitch + i] = to_storage<T>(norm_value(n0, xr[i], inv, i));
        if (h1 != nullptr) h1[size_t(t) * pitch + i] = to_storage<T>(norm_value(n1, xr[i], inv, i));
    }
}

// x = norm(embed[token]), also written to `first` (the first of the vectors that depth averages run over; may be nullptr), and h = next(x)
template <typename T>
__global__ void __launch_bounds__(256) embed_norm_kernel(const T* embed, int pitch, const uint32_t* tokens, int width, float eps, NormParams norm, float* x, float* first, NormParams next, T* h) {
    extern __shared__ float act_smem[];
    __shared__ float red[8];
    const int t = blockIdx.x;
    const T* row = embed + size_t(tokens[t]) * pitch;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
        const float v = from_storage(row[i]);
        act_smem[i] = v, ss += v * v;
    }
    float inv = norm.b == nullptr ? 1.0f / sqrtf(block_sum(ss, red) / static_cast<float>(width) + eps) : 1.0f;
    ss = 0.0f;
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
        const float v = norm_value(norm, act_smem[i], inv, i);
        act_smem[i] = v, ss += v * v;
        x[size_t(t) * width + i] = v;
        if (first != nullptr) first[size_t(t) * width + i] = v;
    }
    if (h == nullptr) return;
    inv = next.b == nullptr ? 1.0f / sqrtf(block_sum(ss, red) / static_cast<float>(width) + eps) : 1.0f;
    for (int i = threadIdx.x; i < width; i += blockDim.x) h[size_t(t) * pitch + i] = to_storage<T>(norm_value(next, act_smem[i], inv, i));
}

// What a layer passes on: x = sum over j < n - 1 of w[j] X_j + w[n - 1] v, where v is the layer's result, stored as X_(n - 1).
struct DepthMix {
    float* x;            // X_j at x + j * stride, each [tokens][width]
    size_t stride;
    const float* w;
    int n;               // 0: the layer's result itself goes on
};

// Rows of the residual stream between the products: v = x + the averaged norms of a pair (PairSum) + the weighted results of the chosen
// experts, then the depth average, then a norm for the next product.
struct RowsArgs {
    const float* x;
    float* x_out;               // may be x
    int width, pitch;
    float eps;
    PairSum pair;
    const void* pick;           // results of the experts [pair rows][width], storage type; nullptr: none
    const uint32_t* pick_row;   // [tokens][top]: their rows
    const float* pick_weight;   // [tokens][top]
    int top;
    DepthMix depth;
    NormParams norm;
    void* h;                    // storage type, [tokens][pitch]; nullptr: no norm
};

template <typename T>
__global__ void __launch_bounds__(256) rows_kernel(const __grid_constant__ RowsArgs a) {
    extern __shared__ float act_smem[];
    __shared__ float red[8];
    __shared__ float2 red2[8];
    const size_t t = blockIdx.x, row = t * a.width;
    const int tid = threadIdx.x;
    float il = 0.0f, ir = 0.0f;
    const bool pair = a.pair.r[0] != nullptr;
    if (pair) {
        float sl = 0.0f, sr = 0.0f;
#pragma unroll 4
        for (int i = tid; i < a.width; i += 256) {
            const float l = a.pair.r[0][row + i], r = a.pair.r[1][row + i];
            sl += l * l, sr += r * r;
        }
        const float2 both = block_sum2(make_float2(sl, sr), red2);
        sl = both.x, sr = both.y;
        il = 0.5f / sqrtf(sl / static_cast<float>(a.width) + a.eps), ir = 0.5f / sqrtf(sr / static_cast<float>(a.width) + a.eps);
    }
    float ss = 0.0f;
    if (a.width % 4 == 0) {  // four elements at a time, every vector's loads together
        const auto at4 = [](const float* p) { return *reinterpret_cast<const float4*>(p); };
        const auto fma4 = [](float f, const float4& x, float4& s) { s.x = fmaf(f, x.x, s.x), s.y = fmaf(f, x.y, s.y), s.z = fmaf(f, x.z, s.z), s.w = fmaf(f, x.w, s.w); };
        for (int i = tid * 4; i < a.width; i += 256 * 4) {
            float4 v = at4(a.x + row + i);
            if (pair) {
                const float4 l = at4(a.pair.r[0] + row + i), r = at4(a.pair.r[1] + row + i), wl = at4(a.pair.w[0] + i), wr = at4(a.pair.w[1] + i);
                v.x += l.x * il * wl.x + r.x * ir * wr.x, v.y += l.y * il * wl.y + r.y * ir * wr.y, v.z += l.z * il * wl.z + r.z * ir * wr.z, v.w += l.w * il * wl.w + r.w * ir * wr.w;
            }
            if (a.pick != nullptr) {
                float4 s = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll 8
                for (int k = 0; k < a.top; ++k) {
                    const T* p = static_cast<const T*>(a.pick) + size_t(a.pick_row[t * a.top + k]) * a.width + i;
                    float4 f;
                    if constexpr (sizeof(T) == 2) {
                        const uint2 u = *reinterpret_cast<const uint2*>(p);
                        f = make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16), __uint_as_float(u.y & 0xffff0000u));
                    } else {
                        f = at4(p);
                    }
                    fma4(a.pick_weight[t * a.top + k], f, s);
                }
                v.x += s.x, v.y += s.y, v.z += s.z, v.w += s.w;
            }
            if (a.depth.n > 0) {
                *reinterpret_cast<float4*>(a.depth.x + (a.depth.n - 1) * a.depth.stride + row + i) = v;
                float4 s = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll 8
                for (int j = 0; j < a.depth.n - 1; ++j) fma4(a.depth.w[j], at4(a.depth.x + j * a.depth.stride + row + i), s);
                fma4(a.depth.w[a.depth.n - 1], v, s);
                v = s;
            }
            if (a.x_out != a.x || pair || a.pick != nullptr || a.depth.n > 0) *reinterpret_cast<float4*>(a.x_out + row + i) = v;
            *reinterpret_cast<float4*>(act_smem + i) = v;
            ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
    } else for (int i = tid; i < a.width; i += 256) {
        float v = a.x[row + i];
        if (pair) v += a.pair.r[0][row + i] * il * a.pair.w[0][i] + a.pair.r[1][row + i] * ir * a.pair.w[1][i];
        if (a.pick != nullptr) {
            float s = 0.0f;
#pragma unroll 4
            for (int k = 0; k < a.top; ++k) s = fmaf(a.pick_weight[t * a.top + k], from_storage(static_cast<const T*>(a.pick)[size_t(a.pick_row[t * a.top + k]) * a.width + i]), s);
            v += s;
        }
        if (a.depth.n > 0) {
            a.depth.x[(a.depth.n - 1) * a.depth.stride + row + i] = v;
            float s = 0.0f;
#pragma unroll 4
            for (int j = 0; j < a.depth.n - 1; ++j) s = fmaf(a.depth.w[j], a.depth.x[j * a.depth.stride + row + i], s);
            v = fmaf(a.depth.w[a.depth.n - 1], v, s);
        }
        a.x_out[row + i] = v;
        act_smem[i] = v, ss += v * v;
    }
    if (a.h == nullptr) return;
    const float inv = a.norm.b == nullptr ? 1.0f / sqrtf(block_sum(ss, red) / static_cast<float>(a.width) + a.eps) : 1.0f;
    __syncthreads();  // (the sums lie in other threads' places)
    for (int i = tid; i < a.width; i += 256) static_cast<T*>(a.h)[t * a.pitch + i] = to_storage<T>(norm_value(a.norm, act_smem[i], inv, i));
}

// The mixer's output norm of many tokens (parts_norm), into the storage type; without a norm a plain conversion. gate (may be nullptr):
// y is first multiplied by silu(gate[token * gate_ld + i]); gate_after: the normed y is (w is then nullptr).
template <typename T>
__global__ void __launch_bounds__(256) finish_rows_kernel(const float* y, const float* gate, const float* gate_after, int gate_ld, int inner, int parts, float eps, const float* w, int w_len, T* out,
                                                          int pitch) {
    extern __shared__ float act_smem[];
    __shared__ float red[8];
    const int t = blockIdx.x;
    for (int i = threadIdx.x; i < inner; i += blockDim.x) {
        const float v = y[size_t(t) * inner + i];
        act_smem[i] = gate != nullptr ? v * silu_f(gate[size_t(t) * gate_ld + i]) : v;
    }
    __syncthreads();
    if (parts > 0 && w != nullptr) parts_norm<float, false>(act_smem, inner, inner, parts, eps, w, w_len, nullptr, red);
    else if (parts > 0) parts_norm<float, true>(act_smem, inner, inner, parts, eps, nullptr, 1, gate_after != nullptr ? gate_after + size_t(t) * gate_ld : nullptr, red);
    for (int i = threadIdx.x; i < inner; i += blockDim.x) out[size_t(t) * pitch + i] = to_storage<T>(act_smem[i]);
}

}  // namespace qtb
