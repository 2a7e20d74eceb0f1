// Mixture of experts over dense (16- or 32-bit) weights, the feed-forward of a layered model's layer. A token's router logits become softmax scores
// over all experts; experts form equal groups of neighbours, only those of the groups with the largest scores can be chosen (a group counts by its
// largest score), and of these the `top` largest are. Their weights are the scores times a factor, not renormalized. A shared expert, which every
// token uses, is multiplied by a number per token; it is projected together with the router (dense_gemv.cuh, dense_gemm_tc.cuh).
//
// One token: moe_up_step_kernel chooses (every block for itself) and makes the chosen experts' activations, moe_down_step_kernel makes their
// results, the residual sum and what follows it. Many tokens: the chosen (token, expert) pairs are sorted by expert, the activations copied in
// that order, and two grouped products run over the experts' runs of rows.
#pragma once
#include "dense_gemm_tc.cuh"

namespace qtb {

struct RouterArgs {
    int experts, groups, keep, top;
    float scale;
};

// One warp: the chosen experts of a token, best first, and their weights, from its logits; equal scores by the lower index. key: 2 * `experts`
// words of shared memory (this warp's). A key is the score's bits plus one (scores are not negative, so their order is that of the bits); 0 stands for
// an expert that cannot be chosen (any more).
__device__ __forceinline__ void choose_experts(const RouterArgs& r, const float* logits, uint32_t* key, int* chosen, float* weight) {
    const int lane = threadIdx.x & 31, size = r.experts / r.groups;
    uint32_t* group = key + r.experts;
    float mx = -INFINITY, sum = 0.0f;
    for (int i = lane; i < r.experts; i += 32) mx = fmaxf(mx, logits[i]);
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    for (int i = lane; i < r.experts; i += 32) {
        const float e = expf(logits[i] - mx);
        key[i] = __float_as_uint(e) + 1u, sum += e;
    }
    sum = warp_sum(sum);
    __syncwarp();
    if (r.keep < r.groups) {  // a group counts by its largest score, and is dropped when `keep` others are better
        for (int g = lane; g < r.groups; g += 32) {
            uint32_t m = 0;
            for (int i = 0; i < size; ++i) m = max(m, key[g * size + i]);
            group[g] = m;
        }
        __syncwarp();
        for (int g = lane; g < r.groups; g += 32) {
            const uint32_t mine = group[g];
            int better = 0;
            for (int o = 0; o < r.groups; ++o) better += group[o] > mine || (group[o] == mine && o < g) ? 1 : 0;
            if (better >= r.keep)
                for (int i = 0; i < size; ++i) key[g * size + i] = 0u;
        }
        __syncwarp();
    }
    uint32_t best = 0;  // this lane's best expert left
    int at = r.experts;
    auto look = [&]() {
        best = 0, at = r.experts;
        for (int i = lane; i < r.experts; i += 32)
            if (key[i] > best) best = key[i], at = i;
    };
    look();
    for (int k = 0; k < r.top; ++k) {
        const uint32_t top = __reduce_max_sync(0xffffffffu, best);
        const int e = min(static_cast<int>(__reduce_min_sync(0xffffffffu, best == top ? static_cast<uint32_t>(at) : 0xffffffffu)), r.experts - 1);  // (in range whatever the logits are)
        if (lane == 0) chosen[k] = e, weight[k] = __uint_as_float(top - 1u) / sum * r.scale;
        if (lane == (e & 31)) {
            key[e] = 0u;
            look();
        }
        __syncwarp();
    }
}

// ---- one token -----------------------------------------------------------------------------------------------------------------------------
struct MoeUpStepArgs {
    RouterArgs router;
    const float* logits;
    const void* h;          // normed input, storage type, [pitch]
    const void* w;          // [experts][rows_pad][pitch]: gate and up rows in turn
    int pitch, rows_pad, ff;
    void* m;                // [top][m_pitch]: silu(gate) * up, storage type
    int m_pitch;
    int* chosen;            // [top]
    float* weight;
};

template <typename T>
__global__ void __launch_bounds__(kProjectThreads, 4) moe_up_step_kernel(const __grid_constant__ MoeUpStepArgs a) {
    extern __shared__ float act_smem[];  // the input, then the router's keys
    __shared__ int chosen[32];
    __shared__ float weight[32];
    const int tid = threadIdx.x, warps = gridDim.x * (kProjectThreads / 32), units = a.router.top * a.ff;
    pdl_trigger();
    pdl_wait();
    if (tid < 32) {
        choose_experts(a.router, a.logits, reinterpret_cast<uint32_t*>(act_smem + a.pitch), chosen, weight);
        if (blockIdx.x == 0 && tid < a.router.top) a.chosen[tid] = chosen[tid], a.weight[tid] = weight[tid];
    }
    else {
        constexpr int kPer = 16 / sizeof(T);
        for (int i = tid - 32; i < a.pitch / kPer; i += kProjectThreads - 32) act_put_storage(act_smem, i, a.pitch, static_cast<const T*>(a.h));
    }
    __syncthreads();
    auto rows_of = [&](int unit) { return static_cast<const T*>(a.w) + (size_t(chosen[unit / a.ff]) * a.rows_pad + 2 * (unit % a.ff)) * a.pitch; };
    RowHead<2> head;
    int unit = blockIdx.x * (kProjectThreads / 32) + (tid >> 5);
    if (unit < units) load_pieces<T, 2>(head, rows_of(unit), a.pitch, tid & 31);
    for (; unit < units; unit += warps) {
        float v[2];
        dot_rows<T, 2>(rows_of(unit), a.pitch, act_smem, head, v);
        if (unit + warps < units) load_pieces<T, 2>(head, rows_of(unit + warps), a.pitch, tid & 31);
        if ((tid & 31) == 0) static_cast<T*>(a.m)[size_t(unit / a.ff) * a.m_pitch + unit % a.ff] = to_storage<T>(silu_f(v[0]) * v[1]);
    }
}

struct MoeDownStepArgs {
    const float* x;         // residual stream before the feed-forward
    float* x_out;
    int width, top;
    const void* m;          // [top][pitch]
    const void* w;          // [experts][rows_pad][pitch]
    int pitch, rows_pad;
    const int* chosen;
    const float* weight;
    const void* shared_m;   // [shared_pitch]
    const void* shared_w;   // [width][shared_pitch]
    int shared_pitch;
    const float* shared_scale;
    DepthMix depth;
    int rows;               // rows of the result per block
};

constexpr int kMoeDownRows = kProjectThreads / 32;  // at most: a warp ends a row

// A block takes a few rows of the result; its warps share the products of these rows with the activations of every chosen expert.
template <typename T>
__global__ void __launch_bounds__(kProjectThreads, 4) moe_down_step_kernel(const __grid_constant__ MoeDownStepArgs a) {
    extern __shared__ float act_smem[];  // activations of the experts, of the shared expert
    __shared__ float part[kMoeDownRows * 33];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, row0 = blockIdx.x * a.rows, rows = min(a.rows, a.width - row0), per = a.top + 1, units = rows * per;
    float* shared_act = act_smem + a.top * a.pitch;
    pdl_trigger();
    if (lane == 0 && warp < rows) l2_prefetch(static_cast<const T*>(a.shared_w) + size_t(row0 + warp) * a.shared_pitch, a.shared_pitch * sizeof(T));
    pdl_wait();
    auto row_of = [&](int unit) {
        const int r = row0 + unit / per, k = unit % per;
        return k < a.top ? static_cast<const T*>(a.w) + (size_t(a.chosen[k]) * a.rows_pad + r) * a.pitch : static_cast<const T*>(a.shared_w) + size_t(r) * a.shared_pitch;
    };
    auto pitch_of = [&](int unit) { return unit % per < a.top ? a.pitch : a.shared_pitch; };
    // what the ending needs, on its way with the first weights
    const int end_row = row0 + warp;
    float x = 0.0f, w = 0.0f, shared_scale = 0.0f, past = 0.0f;
    if (warp < rows) {
        x = a.x[end_row], shared_scale = *a.shared_scale;
        if (lane < a.top) w = a.weight[lane];
        for (int j = lane; j < a.depth.n - 1; j += 32) past = fmaf(a.depth.w[j], a.depth.x[j * a.depth.stride + end_row], past);
    }
    constexpr int kPer = 16 / sizeof(T), kWarps = kProjectThreads / 32;
    // a warp takes two (row, expert) products at a time
    struct Two { uint4 v[2][4]; };
    auto load = [&](int unit, int p0, Two& b) {
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const int u = unit + k * kWarps;
            const T* row = u < units ? row_of(u) : nullptr;
            const int pieces = u < units ? pitch_of(u) / kPer : 0;
#pragma unroll
            for (int i = 0; i < 4; ++i) b.v[k][i] = p0 + 32 * i < pieces ? load_stream(row + size_t(p0 + 32 * i) * kPer) : make_uint4(0, 0, 0, 0);
        }
    };
    Two now;
    load(warp, lane, now);
    for (int i = tid; i < a.top * (a.pitch / kPer); i += kProjectThreads) {
        const int k = i / (a.pitch / kPer), p = i % (a.pitch / kPer);
        act_put_storage(act_smem + k * a.pitch, p, a.pitch, static_cast<const T*>(a.m) + size_t(k) * a.pitch);
    }
    for (int i = tid; i < a.shared_pitch / kPer; i += kProjectThreads) act_put_storage(shared_act, i, a.shared_pitch, static_cast<const T*>(a.shared_m));
    __syncthreads();
    const int longest = max(a.pitch, a.shared_pitch) / kPer;
    for (int unit = warp; unit < units; unit += 2 * kWarps) {
        float sum[2] = {0.0f, 0.0f};
        for (int p0 = lane; p0 - lane < longest; p0 += 128) {
            if (p0 != lane || unit != warp) load(unit, p0, now);
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                const int u = unit + k * kWarps;
                if (u >= units) continue;
                const int e = u % per, pitch = e < a.top ? a.pitch : a.shared_pitch;
                const float* act = e < a.top ? act_smem + e * a.pitch : shared_act;
#pragma unroll
                for (int i = 0; i < 4; ++i)
                    if (p0 + 32 * i < pitch / kPer) sum[k] += dot_piece(now.v[k][i], act, p0 + 32 * i, pitch, T());
            }
        }
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const int u = unit + k * kWarps;
            sum[k] = warp_sum(sum[k]);
            if (lane == 0 && u < units) part[u / per * 33 + u % per] = sum[k];
        }
    }
    __syncthreads();
    if (warp < rows) {
        float s = lane < a.top ? part[warp * 33 + lane] * w : 0.0f;
        s = warp_sum(s), past = warp_sum(past);
        if (lane == 0) {
            const float v = x + s + part[warp * 33 + a.top] * shared_scale;
            if (a.depth.n > 0) a.depth.x[(a.depth.n - 1) * a.depth.stride + end_row] = v;
            a.x_out[end_row] = a.depth.n > 0 ? fmaf(a.depth.w[a.depth.n - 1], v, past) : v;
        }
    }
}

// ---- many tokens ---------------------------------------------------------------------------------------------------------------------------
struct MoeRouteArgs {
    RouterArgs router;
    int tokens;
    const float* logits;    // [tokens][experts]
    int* chosen;            // [tokens][top]
    float* weight;          // [tokens][top]
    int* count;             // [experts], zero between launches: tokens of an expert
    int* rank;              // [tokens][top]: a pair's place among those of its expert
    int* first;             // [experts]: first pair row of an expert
    uint32_t* row;          // [tokens][top]: row of a pair
    DenseRun *up_runs, *down_runs;
    int *n_runs;
    int up_rows, down_rows, tile;  // weight rows of an expert in the two stacks; activation rows of a run
};

// A warp per token. dynamic shared memory: 8 * experts words
__global__ void __launch_bounds__(128) moe_route_kernel(const __grid_constant__ MoeRouteArgs a) {
    extern __shared__ uint32_t route_sm[];
    __shared__ int chosen[4][32];
    __shared__ float weight[4][32];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x * 4 + warp, top = a.router.top;
    if (t >= a.tokens) return;
    choose_experts(a.router, a.logits + size_t(t) * a.router.experts, route_sm + warp * 2 * a.router.experts, chosen[warp], weight[warp]);
    __syncwarp();
    if (lane < top) {
        const int e = chosen[warp][lane];
        a.chosen[t * top + lane] = e, a.weight[t * top + lane] = weight[warp][lane];
        a.rank[t * top + lane] = atomicAdd(a.count + e, 1);
    }
}

// One block of 1024 threads, a thread per expert: where the experts' rows begin, and the runs of both products. Leaves the counts at zero.
__global__ void __launch_bounds__(1024) moe_plan_kernel(const __grid_constant__ MoeRouteArgs a) {
    __shared__ int rows_sum[32], runs_sum[32];
    const int e = threadIdx.x, warp = e >> 5, lane = e & 31;
    const int n = e < a.router.experts ? a.count[e] : 0, r = (n + a.tile - 1) / a.tile;
    int rows = n, runs = r;  // running sums
    for (int o = 1; o < 32; o <<= 1) {
        const int x = __shfl_up_sync(0xffffffffu, rows, o), y = __shfl_up_sync(0xffffffffu, runs, o);
        if (lane >= o) rows += x, runs += y;
    }
    if (lane == 31) rows_sum[warp] = rows, runs_sum[warp] = runs;
    __syncthreads();
    int rows0 = 0, runs0 = 0, all = 0;
    for (int w = 0; w < 32; ++w) {
        if (w < warp) rows0 += rows_sum[w], runs0 += runs_sum[w];
        all += runs_sum[w];
    }
    rows0 += rows - n, runs0 += runs - r;
    if (e == 0) *a.n_runs = all;
    if (e >= a.router.experts) return;
    a.first[e] = rows0, a.count[e] = 0;
    for (int k = 0; k < r; ++k) {
        const int from = k * a.tile, here = min(a.tile, n - from);
        a.up_runs[runs0 + k] = DenseRun{e * a.up_rows, rows0 + from, here, 0};
        a.down_runs[runs0 + k] = DenseRun{e * a.down_rows, rows0 + from, here, 0};
    }
}

// Copies each pair's activations to its row. grid: (top, tokens); pitch in 16-byte pieces
__global__ void __launch_bounds__(128) moe_gather_kernel(const __grid_constant__ MoeRouteArgs a, const uint4* h, uint4* out, int pieces) {
    const int pair = blockIdx.y * a.router.top + blockIdx.x;
    const uint32_t row = a.first[a.chosen[pair]] + a.rank[pair];
    if (threadIdx.x == 0) a.row[pair] = row;
    for (int i = threadIdx.x; i < pieces; i += 128) out[size_t(row) * pieces + i] = h[size_t(blockIdx.y) * pieces + i];
}

}  // namespace qtb
