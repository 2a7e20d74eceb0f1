// Dense projections of many tokens: out[t][r] = sum_k W[r][k] * h[t][k], with the endings of dense_gemv.cuh.
//
// 16-bit weights run on the 5th-generation tensor cores. A tile is 128 weight rows (the M of the instruction) x 128 or 256 tokens (the N):
// one thread fetches 64-column slices of both operands with TMA (128-byte swizzle) into a ring of stages, one thread issues
// tcgen05.mma.kind::f16 (bf16 operands, 32-bit sums in tensor memory), eight warps read the sums with tcgen05.ld - a weight row per lane, so
// that the 32 lanes of a warp write 32 neighbouring results of a token - and apply the ending. One block per multiprocessor takes tiles in
// turn; two sets of accumulators let the ending of a tile overlap the products of the next. Tiles run over the tokens first, so the blocks
// that are at work together share weight rows.
//
// The dual form makes two products of one tile, W_o y and W_down m, in two accumulators and ends with both gates and the residual sum.
// The grouped form multiplies runs of consecutive activation rows, each with its own range of weight rows (the experts of a mixture); which
// runs there are is read from device memory.
// Every wait is bounded, as in gemm_tc.cuh, whose mbarrier, descriptor and status conventions are used here.
//
// 32-bit weights: a plain tiled kernel in 32-bit arithmetic with the same endings.
#pragma once
#include <cuda.h>

#include "dense_gemv.cuh"
#include "gemm_tc.cuh"

namespace qtb {

constexpr int kDenseM = 128, kDenseBox = 128, kDenseK = 64;  // kDenseBox: rows of an activation box; a tile's N is a multiple of it
constexpr int kDenseEndWarps = 8;
constexpr int kDenseThreads = 64 + 32 * kDenseEndWarps;  // TMA warp, MMA warp, warps for the ending
__host__ __device__ constexpr int dense_stages(int n) { return n > 128 ? 4 : 6; }
__host__ __device__ constexpr int dense_stage_bytes(int n) { return (kDenseM + n) * kDenseK * 2; }
__host__ __device__ constexpr int dense_smem(int n) { return dense_stages(n) * dense_stage_bytes(n) + 1024 + 256; }

enum DenseForm : int { kDensePlain = 0, kDenseDual = 1, kDenseGrouped = 2 };
// Grouped form: activation rows token0 .. token0 + tokens - 1 (at most a tile's N) times the weight rows from row0 on.
struct DenseRun { int row0, token0, tokens, pad; };

struct DenseGemmArgs {
    int tokens;
    int n_prob;              // plain form: 1 or 2 stacks, each over its own activations
    int k_steps[2];          // 64-column slices
    int row_tiles[2];        // grouped form: of one range of weight rows
    DenseStack stack[2];     // plain and grouped form: the endings
    // dual form
    float* x;
    int width;
    const float *gate1, *gate2;
    const float* token_gate;      // factor of the first product, one per token; nullptr: 1
    // grouped form
    const DenseRun* runs;
    const int* n_runs;
    unsigned int* status;
    unsigned int spin_limit;
};

// One result of a plain-form tile. `pair` is the neighbouring row's value (SwiGLU: rows 2 i and 2 i + 1 are gate and up of channel i).
template <typename T>
__device__ __forceinline__ void dense_end(const DenseSeg& g, int row, int token, float v, float pair) {
    if (row >= g.rows) return;
    if (g.kind == kSegSwiGlu) {
        if ((row & 1) == 0) static_cast<T*>(g.t)[size_t(token) * g.ld + (row >> 1)] = to_storage<T>(silu_f(v) * pair);
    } else if (g.kind == kSegStore) {
        static_cast<T*>(g.t)[size_t(token) * g.ld + row] = to_storage<T>(v);
    } else {
        g.f[size_t(token) * g.ld + row] = g.kind == kSegSigmoid ? sigmoid_f(v + (g.bias != nullptr ? g.bias[row] : 0.0f)) : v;
    }
}

// Sixteen results of a weight row, tokens `token` .. token + n - 1 (n <= 16), of a plain- or grouped-form tile in 16-bit storage. Lanes 2 i and
// 2 i + 1 hold rows 2 i and 2 i + 1: where both rows end up beside one another, each of the two lanes takes eight tokens for both.
__device__ __forceinline__ void dense_end16(const DenseSeg& g, int row, int token, int n, const uint32_t (&v)[16]) {
    const int kind = g.kind, lane = threadIdx.x & 31;
    const size_t ld = g.ld;
    if (kind == kSegPlain || kind == kSegSigmoid) {
        if (row >= g.rows) return;
        float* f = g.f + size_t(token) * ld + row;
        if (kind == kSegPlain) {
            if (n >= 16) {
#pragma unroll
                for (int i = 0; i < 16; ++i) f[i * ld] = __uint_as_float(v[i]);
            } else {
#pragma unroll
                for (int i = 0; i < 16; ++i)
                    if (i < n) f[i * ld] = __uint_as_float(v[i]);
            }
            return;
        }
        const float bias = g.bias != nullptr ? g.bias[row] : 0.0f;
#pragma unroll
        for (int i = 0; i < 16; ++i)
            if (i < n) f[i * ld] = sigmoid_f(__uint_as_float(v[i]) + bias);
        return;
    }
    const bool odd = lane & 1;
    float a[8], b[8];  // of rows 2 i and 2 i + 1, the first or the last eight tokens
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const uint32_t other = __shfl_xor_sync(0xffffffffu, odd ? v[i] : v[i + 8], 1);
        a[i] = __uint_as_float(odd ? other : v[i]), b[i] = __uint_as_float(odd ? v[i + 8] : other);
    }
    const int mine = odd ? 8 : 0, even = row & ~1;
    if (even >= g.rows) return;
    bf16* t = static_cast<bf16*>(g.t) + size_t(token + mine) * ld;
    if (kind == kSegSwiGlu) {
        t += even >> 1;
#pragma unroll
        for (int i = 0; i < 8; ++i)
            if (mine + i < n) t[i * ld] = __float2bfloat16_rn(__fdividef(a[i], 1.0f + __expf(-a[i])) * b[i]);
        return;
    }
    t += even;
    if (ld % 2 == 0 && even + 1 < g.rows) {
#pragma unroll
        for (int i = 0; i < 8; ++i)
            if (mine + i < n) *reinterpret_cast<__nv_bfloat162*>(t + i * ld) = __floats2bfloat162_rn(a[i], b[i]);
        return;
    }
#pragma unroll
    for (int i = 0; i < 8; ++i)
        if (mine + i < n) {
            t[i * ld] = __float2bfloat16_rn(a[i]);
            if (even + 1 < g.rows) t[i * ld + 1] = __float2bfloat16_rn(b[i]);
        }
}

namespace dense_detail {
__device__ __forceinline__ void tma_load_2d(uint32_t dst, const CUtensorMap* map, int x, int y, uint32_t bar) {
    asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(dst), "l"(map), "r"(x), "r"(y), "r"(bar) : "memory");
}
// kind::f16 with bf16 operands: F32 accumulator (1 at bit 4), BF16 A and B (1 at bits 7 and 10), both K-major, N / 8 at bit 17, M / 16 at bit 24.
__device__ __forceinline__ uint32_t instr_desc_bf16(int m, int n) { return (1u << 4) | (1u << 7) | (1u << 10) | (uint32_t(n >> 3) << 17) | (uint32_t(m >> 4) << 24); }
__device__ __forceinline__ void mma_bf16(uint32_t tmem_d, uint64_t desc_a, uint64_t desc_b, uint32_t idesc, uint32_t accumulate) {
    const uint32_t zero = 0;  // no output lane is disabled
    asm volatile(
        "{\n\t.reg .pred p;\n\t"
        "setp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, {%5, %5, %5, %5}, p;\n\t}" ::"r"(tmem_d),
        "l"(desc_a), "l"(desc_b), "r"(idesc), "r"(accumulate), "r"(zero)
        : "memory");
}
__device__ __forceinline__ void tmem_load16(uint32_t taddr, uint32_t (&v)[16]) {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];"
        : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]), "=r"(v[8]), "=r"(v[9]), "=r"(v[10]), "=r"(v[11]), "=r"(v[12]), "=r"(v[13]),
          "=r"(v[14]), "=r"(v[15])
        : "r"(taddr));
}
}  // namespace dense_detail

template <int N, int FORM>
__global__ void __launch_bounds__(kDenseThreads, 1) dense_gemm_tc_kernel(const __grid_constant__ CUtensorMap w0, const __grid_constant__ CUtensorMap h0, const __grid_constant__ CUtensorMap w1,
                                                                         const __grid_constant__ CUtensorMap h1, const __grid_constant__ DenseGemmArgs a) {
    using namespace gemm_detail;
    using namespace dense_detail;
    constexpr bool DUAL = FORM == kDenseDual, GROUPED = FORM == kDenseGrouped;
    extern __shared__ unsigned char dense_smem_raw[];
    unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(dense_smem_raw) + 1023) & ~uintptr_t(1023));
    constexpr int S = dense_stages(N), kStage = dense_stage_bytes(N), kAcc = DUAL ? 2 * N : N;  // kAcc: tensor-memory columns of a tile
    static_assert(2 * kAcc <= 512, "two sets of accumulators fit tensor memory");
    uint64_t* bars = reinterpret_cast<uint64_t*>(smem + S * kStage);
    const uint32_t bar0 = smem_u32(bars), tiles0 = smem_u32(smem);
    auto loaded = [&](int s) { return bar0 + 8u * s; };
    auto empty = [&](int s) { return bar0 + 8u * (S + s); };
    auto acc_full = [&](int i) { return bar0 + 8u * (2 * S + i); };
    auto acc_empty = [&](int i) { return bar0 + 8u * (2 * S + 2 + i); };
    volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(bars + 2 * S + 4);
    volatile unsigned int* abort_flag = reinterpret_cast<volatile unsigned int*>(bars + 2 * S + 5);

    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int token_tiles = (a.tokens + N - 1) / N;
    const int items = GROUPED ? *a.n_runs * a.row_tiles[0] : token_tiles * (a.row_tiles[0] + (!DUAL && a.n_prob > 1 ? a.row_tiles[1] : 0));
    // tile `item`: its problem, first row and first token
    auto locate = [&](int item, int* prob, int* row0, int* token0) {
        if constexpr (GROUPED) {
            const DenseRun run = a.runs[item / a.row_tiles[0]];
            *prob = 0, *row0 = run.row0 + item % a.row_tiles[0] * kDenseM, *token0 = run.token0;
            return;
        }
        const int tile = item / token_tiles;
        *prob = !DUAL && tile >= a.row_tiles[0] ? 1 : 0;
        *row0 = (tile - (*prob ? a.row_tiles[0] : 0)) * kDenseM;
        *token0 = (item % token_tiles) * N;
    };

    if (tid == 0) {
        for (int s = 0; s < S; ++s) {
            mbar_init(loaded(s), 1);
            mbar_init(empty(s), 1);
        }
        for (int i = 0; i < 2; ++i) {
            mbar_init(acc_full(i), 1);
            mbar_init(acc_empty(i), kDenseEndWarps);
        }
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 0) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(const_cast<uint32_t*>(tmem_slot))), "r"(512u) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem_base = *tmem_slot;

    if (warp == 0) {
        if (lane == 0) {
            int it = 0, s = 0;
            uint32_t ph = 0;
            bool okay = true;
            for (int item = blockIdx.x; item < items && okay; item += gridDim.x) {
                int prob, row0, token0;
                locate(item, &prob, &row0, &token0);
                const int steps0 = a.k_steps[prob], steps = DUAL ? steps0 + a.k_steps[1] : steps0;
                for (int k = 0; k < steps; ++k, ++it) {
                    if (!(okay = mbar_wait(empty(s), ph ^ 1, abort_flag, a.spin_limit))) break;
                    const bool second = DUAL ? k >= steps0 : prob != 0;
                    const int x = (DUAL && second ? k - steps0 : k) * kDenseK;
                    const uint32_t dst = tiles0 + s * kStage;
                    mbar_expect_tx(loaded(s), kStage);
                    tma_load_2d(dst, second ? &w1 : &w0, x, row0, loaded(s));
#pragma unroll
                    for (int b = 0; b < N / kDenseBox; ++b)
                        tma_load_2d(dst + (kDenseM + b * kDenseBox) * kDenseK * 2, second ? &h1 : &h0, x, token0 + b * kDenseBox, loaded(s));
                    if (++s == S) s = 0, ph ^= 1;
                }
            }
            for (int back = 0; back < min(it, S); ++back) {  // its copies in flight land before the block leaves
                if (--s < 0) s = S - 1, ph ^= 1;
                mbar_wait(loaded(s), ph, abort_flag, a.spin_limit, false);
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t idesc = instr_desc_bf16(kDenseM, N);
            int s = 0, j = 0;
            uint32_t ph = 0;
            bool okay = true;
            for (int item = blockIdx.x; item < items && okay; item += gridDim.x, ++j) {
                int prob, row0, token0;
                locate(item, &prob, &row0, &token0);
                const int steps0 = a.k_steps[prob], steps = DUAL ? steps0 + a.k_steps[1] : steps0;
                const int set = j & 1;
                if (!(okay = mbar_wait(acc_empty(set), ((j >> 1) & 1) ^ 1, abort_flag, a.spin_limit))) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                for (int k = 0; k < steps; ++k) {
                    if (!(okay = mbar_wait(loaded(s), ph, abort_flag, a.spin_limit))) break;
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                    const uint32_t at = tiles0 + s * kStage;
                    const uint64_t da = smem_desc(at, 16, 1024, 2), db = smem_desc(at + kDenseM * kDenseK * 2, 16, 1024, 2);  // 128-byte swizzle, 8-row groups 1024 bytes apart
                    const uint32_t acc = tmem_base + set * kAcc + (DUAL && k >= steps0 ? N : 0);
                    const bool first = k == 0 || (DUAL && k == steps0);
#pragma unroll
                    for (int q = 0; q < kDenseK / 16; ++q) mma_bf16(acc, da + 2 * q, db + 2 * q, idesc, first && q == 0 ? 0u : 1u);
                    mma_commit(empty(s));
                    if (++s == S) s = 0, ph ^= 1;
                }
                mma_commit(acc_full(set));  // (also on the way out after a failed wait)
            }
        }
    } else {
        // the ending: a warp reads the 32 lanes of tensor memory that its index modulo 4 selects; the two warps of a quarter take 16-column pieces in turn
        const int r = (warp & 3) * 32 + lane, turn = (warp - 2) >> 2;
        int j = 0;
        for (int item = blockIdx.x; item < items; item += gridDim.x, ++j) {
            int prob, row0, token0;
            locate(item, &prob, &row0, &token0);
            const int set = j & 1;
            bool okay = true;
            if (lane == 0) okay = mbar_wait(acc_full(set), (j >> 1) & 1, abort_flag, a.spin_limit) && *abort_flag == 0;
            okay = __shfl_sync(0xffffffffu, okay ? 1 : 0, 0) != 0;
            if (!okay) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const uint32_t acc = tmem_base + (uint32_t((warp & 3) * 32) << 16) + set * kAcc;
            const int n_here = GROUPED ? a.runs[item / a.row_tiles[0]].tokens : min(N, a.tokens - token0);
            if constexpr (DUAL) {
                const int row = row0 + r;
                const bool has2 = a.k_steps[1] > 0;
                for (int c0 = turn * 16; c0 < n_here; c0 += 32) {
                    uint32_t v1[16], v2[16];
                    tmem_load16(acc + c0, v1);
                    if (has2) tmem_load16(acc + N + c0, v2);
                    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
                    if (row < a.width) {
                        const size_t at = size_t(token0 + c0) * a.width + row;
                        const int n16 = min(16, n_here - c0);
                        float add[16], x[16];
#pragma unroll
                        for (int i = 0; i < 16; ++i) {
                            x[i] = i < n16 ? a.x[at + i * size_t(a.width)] : 0.0f;
                            add[i] = __uint_as_float(v1[i]);
                        }
                        if (a.gate1 != nullptr) {
#pragma unroll
                            for (int i = 0; i < 16; ++i) add[i] *= i < n16 ? a.gate1[at + i * size_t(a.width)] : 0.0f;
                        } else if (a.token_gate != nullptr) {
#pragma unroll
                            for (int i = 0; i < 16; ++i) add[i] *= i < n16 ? a.token_gate[token0 + c0 + i] : 0.0f;
                        }
                        if (has2) {
                            if (a.gate2 != nullptr) {
#pragma unroll
                                for (int i = 0; i < 16; ++i) add[i] = fmaf(__uint_as_float(v2[i]), i < n16 ? a.gate2[at + i * size_t(a.width)] : 0.0f, add[i]);
                            } else {
#pragma unroll
                                for (int i = 0; i < 16; ++i) add[i] += __uint_as_float(v2[i]);
                            }
                        }
#pragma unroll
                        for (int i = 0; i < 16; ++i)
                            if (i < n16) a.x[at + i * size_t(a.width)] = x[i] + add[i];
                    }
                }
            } else {
                const DenseStack& st = a.stack[prob];
                const int stack_row0 = GROUPED ? row0 - a.runs[item / a.row_tiles[0]].row0 : row0;
                const DenseSeg& g = dense_seg_of(st, stack_row0);
                for (int c0 = turn * 32; c0 < n_here; c0 += 64) {  // (the columns behind n_here exist: N is a multiple of 64)
                    uint32_t v[2][16];
                    tmem_load16(acc + c0, v[0]);
                    tmem_load16(acc + c0 + 16, v[1]);
                    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
                    dense_end16(g, stack_row0 + r - g.row0, token0 + c0, n_here - c0, v[0]);
                    if (c0 + 16 < n_here) dense_end16(g, stack_row0 + r - g.row0, token0 + c0 + 16, n_here - c0 - 16, v[1]);
                }
            }
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            __syncwarp();
            if (lane == 0) mbar_arrive(acc_empty(set));
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (tid == 0 && *abort_flag) atomicExch(a.status, kGemmStatusTimeout);
    if (warp == 0) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(512u) : "memory");
    }
}

// ---- 32-bit products ------------------------------------------------------------------------------------------------------------------
constexpr int kF32Tile = 64, kF32K = 16;

template <int FORM>
__global__ void __launch_bounds__(256) dense_gemm_f32_kernel(const float* w0, const float* h0, int pitch0, const float* w1, const float* h1, int pitch1, const __grid_constant__ DenseGemmArgs a) {
    constexpr bool DUAL = FORM == kDenseDual, GROUPED = FORM == kDenseGrouped;
    __shared__ float ws[kF32K][kF32Tile + 4], hs[kF32K][kF32Tile + 4];
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int per = kDenseM / kF32Tile;  // row tiles are counted in units of kDenseM
    if (GROUPED && static_cast<int>(blockIdx.x) >= *a.n_runs) return;
    const DenseRun run = GROUPED ? a.runs[blockIdx.x] : DenseRun{0, static_cast<int>(blockIdx.x) * kF32Tile, 0, 0};
    const int token0 = run.token0, end = GROUPED ? token0 + run.tokens : a.tokens;
    const int prob = !DUAL && !GROUPED && static_cast<int>(blockIdx.y) >= a.row_tiles[0] * per ? 1 : 0;
    const int row0 = (static_cast<int>(blockIdx.y) - (prob ? a.row_tiles[0] * per : 0)) * kF32Tile;
    float acc[2][4][4] = {};
    for (int half = 0; half < (DUAL ? 2 : 1); ++half) {
        const bool second = DUAL ? half == 1 : prob != 0;
        const float *w = second ? w1 : w0, *h = second ? h1 : h0;
        const int pitch = second ? pitch1 : pitch0, k_end = a.k_steps[second ? 1 : 0] * kDenseK;
        for (int k0 = 0; k0 < k_end; k0 += kF32K) {
            __syncthreads();
            for (int i = tid; i < kF32Tile * kF32K; i += 256) {
                const int r = i / kF32K, k = i % kF32K;
                ws[k][r] = w[size_t(run.row0 + row0 + r) * pitch + k0 + k];
                hs[k][r] = token0 + r < end ? h[size_t(token0 + r) * pitch + k0 + k] : 0.0f;
            }
            __syncthreads();
#pragma unroll
            for (int k = 0; k < kF32K; ++k) {
                float wv[4], hv[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) wv[i] = ws[k][tx * 4 + i], hv[i] = hs[k][ty * 4 + i];
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int j = 0; j < 4; ++j) acc[half][i][j] = fmaf(wv[i], hv[j], acc[half][i][j]);
            }
        }
    }
    for (int j = 0; j < 4; ++j) {
        const int token = token0 + ty * 4 + j;
        if (token >= end) continue;
        for (int i = 0; i < 4; ++i) {
            const int row = row0 + tx * 4 + i;
            if constexpr (DUAL) {
                if (row >= a.width) continue;
                const size_t at = size_t(token) * a.width + row;
                float add = acc[0][i][j];
                if (a.gate1 != nullptr) add *= a.gate1[at];
                else if (a.token_gate != nullptr) add *= a.token_gate[token];
                if (a.k_steps[1] > 0) add += acc[1][i][j] * (a.gate2 != nullptr ? a.gate2[at] : 1.0f);
                a.x[at] += add;
            } else {
                const DenseStack& st = a.stack[prob];
                const DenseSeg& g = dense_seg_of(st, row0);
                dense_end<float>(g, row - g.row0, token, acc[0][i][j], acc[0][i ^ 1][j]);
            }
        }
    }
}

}  // namespace qtb
