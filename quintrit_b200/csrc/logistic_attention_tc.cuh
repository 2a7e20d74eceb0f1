// The attention of logistic_attention.cuh for many query tokens on the 5th-generation tensor cores: 128 query positions of one head per block, keys
// and values in tiles of 128, heads of up to 128 dimensions.
//
//   * one thread fetches the queries once and then keys and values of tile after tile with TMA (64-column slices, 128-byte swizzle) into three stages;
//   * one thread issues S = Q K^T (both operands from shared memory) into one of two score areas of tensor memory and, a tile behind,
//     O += P V with P from tensor memory and V as it lies in the cache - rows are keys, so it is the operand whose N runs fastest;
//   * sixteen warps make the weights: a query row per lane (a warp reaches the 32 lanes that its index modulo 4 selects, four warps share them by
//     columns), read with tcgen05.ld, written back as bf16 pairs over the scores they came from with tcgen05.st. A weight depends on its own score
//     alone: nothing is rescaled, O stays in tensor memory until the end.
//
// Products of the same thread run in the order in which they are issued, so the scores of tile j + 1 may take the place of the weights of tile j - 1
// once their product is issued. Two weights share one reciprocal (of the product of their denominators; exponents are held at 62 so that it
// stays finite). Every wait is bounded, as in gemm_tc.cuh, whose mbarrier, descriptor and status conventions are used here.
#pragma once
#include "dense_gemm_tc.cuh"
#include "logistic_attention.cuh"

namespace qtb {

constexpr int kLtRows = 128, kLtKeys = 128, kLtStages = 3;
constexpr int kLtWeightWarps = 16, kLtThreads = 64 + 32 * kLtWeightWarps;  // TMA warp, MMA warp, weight warps
constexpr int kLtSlice = kLtKeys * 64 * 2;                                // bytes of a 64-column slice of 128 rows

inline int logistic_tc_slices(int dim) { return (dim + 63) / 64; }
inline bool logistic_tc_fits(int dim, int vdim) { return dim <= 128 && vdim <= 128; }
inline size_t logistic_tc_smem(int dim, int vdim) {
    const size_t k = logistic_tc_slices(dim), v = logistic_tc_slices(vdim);
    return (k + kLtStages * (k + v)) * kLtSlice + 1024 + 256;
}

struct LogisticTcArgs {
    LogisticArgs a;
    int k_slices, v_slices;
    int slot;                 // the sequence's, in the cache
    unsigned int* status;
    unsigned int spin_limit;
};

__device__ __forceinline__ float fast_reciprocal(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

namespace dense_detail {
__device__ __forceinline__ void mma_bf16_ts(uint32_t tmem_d, uint32_t tmem_a, uint64_t desc_b, uint32_t idesc, uint32_t accumulate) {
    const uint32_t zero = 0;
    asm volatile(
        "{\n\t.reg .pred p;\n\t"
        "setp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, {%5, %5, %5, %5}, p;\n\t}" ::"r"(tmem_d),
        "r"(tmem_a), "l"(desc_b), "r"(idesc), "r"(accumulate), "r"(zero)
        : "memory");
}
__device__ __forceinline__ void tmem_store16(uint32_t taddr, const uint32_t (&v)[16]) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};" ::"r"(taddr), "r"(v[0]), "r"(v[1]), "r"(v[2]),
        "r"(v[3]), "r"(v[4]), "r"(v[5]), "r"(v[6]), "r"(v[7]), "r"(v[8]), "r"(v[9]), "r"(v[10]), "r"(v[11]), "r"(v[12]), "r"(v[13]), "r"(v[14]), "r"(v[15])
        : "memory");
}
}  // namespace dense_detail

// grid: (query tiles, heads); the last tiles, which see most keys, come first
__global__ void __launch_bounds__(kLtThreads, 1) logistic_tc_kernel(const __grid_constant__ CUtensorMap qmap, const __grid_constant__ CUtensorMap kmap, const __grid_constant__ CUtensorMap vmap,
                                                                    const __grid_constant__ LogisticTcArgs t) {
    using namespace gemm_detail;
    using namespace dense_detail;
    extern __shared__ unsigned char lt_raw[];
    const LogisticArgs& a = t.a;
    unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(lt_raw) + 1023) & ~uintptr_t(1023));
    const int ks = t.k_slices, vs = t.v_slices;
    const uint32_t q_tile = smem_u32(smem), stage0 = q_tile + ks * kLtSlice, stage_bytes = (ks + vs) * kLtSlice;
    uint64_t* bars = reinterpret_cast<uint64_t*>(smem + (ks + kLtStages * (ks + vs)) * kLtSlice);
    const uint32_t bar0 = smem_u32(bars);
    const uint32_t q_loaded = bar0, o_full = bar0 + 8;
    auto k_loaded = [&](int s) { return bar0 + 16u + 8u * s; };
    auto v_loaded = [&](int s) { return bar0 + 40u + 8u * s; };
    auto k_empty = [&](int s) { return bar0 + 64u + 8u * s; };
    auto v_empty = [&](int s) { return bar0 + 88u + 8u * s; };
    auto s_full = [&](int i) { return bar0 + 112u + 8u * i; };
    auto p_full = [&](int i) { return bar0 + 128u + 8u * i; };
    static_assert(kLtStages == 3, "places of the barriers");
    volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(bars + 18);
    volatile unsigned int* abort_flag = reinterpret_cast<volatile unsigned int*>(bars + 19);

    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int head = blockIdx.y, kvh = head / (a.heads / a.kv_heads), q0 = (gridDim.x - 1 - blockIdx.x) * kLtRows;
    const int pos0 = static_cast<int>(seq_position(a.seq, a.pos, 0));
    const int first = pos0 + q0, last = pos0 + min(q0 + kLtRows, a.tokens) - 1, tiles = last / kLtKeys + 1;

    if (tid == 0) {
        mbar_init(q_loaded, 1), mbar_init(o_full, 1);
        for (int s = 0; s < kLtStages; ++s) mbar_init(k_loaded(s), 1), mbar_init(v_loaded(s), 1), mbar_init(k_empty(s), 1), mbar_init(v_empty(s), 1);
        for (int i = 0; i < 2; ++i) mbar_init(s_full(i), 1), mbar_init(p_full(i), kLtWeightWarps);
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
    const uint32_t tmem = *tmem_slot, o_acc = tmem + 2 * kLtKeys;  // scores (and weights) of two tiles, then the output

    if (warp == 0) {
        if (lane == 0) {
            mbar_expect_tx(q_loaded, ks * kLtSlice);
            for (int i = 0; i < ks; ++i) tma_load_2d(q_tile + i * kLtSlice, &qmap, (head * ks + i) * 64, q0, q_loaded);
            int keys = 0, values = 0;  // tiles asked for
            for (int tile = 0; tile < tiles; ++tile) {
                const int s = tile % kLtStages;
                const uint32_t dst = stage0 + s * stage_bytes, parity = ((tile / kLtStages) & 1) ^ 1;
                if (!mbar_wait(k_empty(s), parity, abort_flag, t.spin_limit)) break;
                mbar_expect_tx(k_loaded(s), ks * kLtSlice);
                for (int i = 0; i < ks; ++i) tma_load_3d(dst + i * kLtSlice, &kmap, kvh * a.dim_pad + i * 64, tile * kLtKeys, t.slot, k_loaded(s));
                ++keys;
                if (!mbar_wait(v_empty(s), parity, abort_flag, t.spin_limit)) break;
                mbar_expect_tx(v_loaded(s), vs * kLtSlice);
                for (int i = 0; i < vs; ++i) tma_load_3d(dst + (ks + i) * kLtSlice, &vmap, kvh * a.vdim_pad + i * 64, tile * kLtKeys, t.slot, v_loaded(s));
                ++values;
            }
            // its copies in flight land before the block leaves
            mbar_wait(q_loaded, 0, abort_flag, t.spin_limit, false);
            for (int k = max(0, keys - kLtStages); k < keys; ++k) mbar_wait(k_loaded(k % kLtStages), (k / kLtStages) & 1, abort_flag, t.spin_limit, false);
            for (int k = max(0, values - kLtStages); k < values; ++k) mbar_wait(v_loaded(k % kLtStages), (k / kLtStages) & 1, abort_flag, t.spin_limit, false);
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t score_desc = instr_desc_bf16(kLtRows, kLtKeys), out_desc = instr_desc_bf16(kLtRows, vs * 64) | (1u << 16);  // bit 16: N runs fastest in B
            auto scores = [&](int tile) {
                const int s = tile % kLtStages;
                if (!mbar_wait(k_loaded(s), (tile / kLtStages) & 1, abort_flag, t.spin_limit)) return false;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                for (int i = 0; i < ks; ++i) {
                    const uint64_t dq = smem_desc(q_tile + i * kLtSlice, 16, 1024, 2), dk = smem_desc(stage0 + s * stage_bytes + i * kLtSlice, 16, 1024, 2);
#pragma unroll
                    for (int q = 0; q < 4; ++q) mma_bf16(tmem + (tile & 1) * kLtKeys, dq + 2 * q, dk + 2 * q, score_desc, i == 0 && q == 0 ? 0u : 1u);
                }
                mma_commit(s_full(tile & 1));
                mma_commit(k_empty(s));
                return true;
            };
            bool okay = mbar_wait(q_loaded, 0, abort_flag, t.spin_limit) && scores(0);
            for (int tile = 0; tile < tiles && okay; ++tile) {
                if (tile + 1 < tiles && !(okay = scores(tile + 1))) break;
                const int s = tile % kLtStages;
                if (!(okay = mbar_wait(p_full(tile & 1), (tile >> 1) & 1, abort_flag, t.spin_limit) && mbar_wait(v_loaded(s), (tile / kLtStages) & 1, abort_flag, t.spin_limit))) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                // slices of 64 columns of V lie kLtSlice apart, groups of eight keys 1024 bytes; the weights of 32 keys begin where their scores did
                const uint64_t dv = smem_desc(stage0 + s * stage_bytes + ks * kLtSlice, kLtSlice, 1024, 2);
#pragma unroll
                for (int k = 0; k < kLtKeys / 16; ++k)
                    mma_bf16_ts(o_acc, tmem + (tile & 1) * kLtKeys + (k >> 1) * 32 + (k & 1) * 8, dv + k * (2048 >> 4), out_desc, tile == 0 && k == 0 ? 0u : 1u);
                mma_commit(v_empty(s));
            }
            mma_commit(o_full);  // (also on the way out after a failed wait)
        }
    } else {
        const int r = (warp & 3) * 32 + lane, part = (warp - 2) >> 2, row = first + r;
        const uint32_t mine = tmem + (uint32_t((warp & 3) * 32) << 16);
        // exp(-score) = exp2(-log2(e) score): the sign and log2(e) go into the factors
        constexpr float kLog2e = 1.4426950408889634f;
        const float scale = -kLog2e * a.scale, slope = kLog2e * a.slope[head], bias = -kLog2e * a.bias[head];
        bool okay = true;
        for (int tile = 0; tile < tiles && okay; ++tile) {
            if (lane == 0) okay = mbar_wait(s_full(tile & 1), (tile >> 1) & 1, abort_flag, t.spin_limit);
            okay = __shfl_sync(0xffffffffu, okay ? 1 : 0, 0) != 0;
            if (!okay) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const uint32_t area = mine + (tile & 1) * kLtKeys + part * 32;
            const int k0 = tile * kLtKeys + part * 32;
            const float base = fmaf(slope, static_cast<float>(row - k0), bias);
            uint32_t v[2][16], p[16];
            tmem_load16(area, v[0]), tmem_load16(area + 16, v[1]);
            asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
            auto weights = [&](bool open) {
#pragma unroll
                for (int i = 0; i < 16; ++i) {
                    const int j = 2 * i;
                    const float x0 = fmaf(__uint_as_float(v[i >> 3][j & 15]), scale, fmaf(-slope, static_cast<float>(j), base));
                    const float x1 = fmaf(__uint_as_float(v[i >> 3][(j + 1) & 15]), scale, fmaf(-slope, static_cast<float>(j + 1), base));
                    const float d0 = 1.0f + fast_exp2(fminf(x0, 62.0f)), d1 = 1.0f + fast_exp2(fminf(x1, 62.0f)), both = fast_reciprocal(d0 * d1);
                    float w0 = both * d1, w1 = both * d0;
                    if (!open) w0 = k0 + j <= row ? w0 : 0.0f, w1 = k0 + j + 1 <= row ? w1 : 0.0f;
                    p[i] = pack_bf16(w0, w1);
                }
            };
            if (k0 + 31 <= first) weights(true);  // every row sees these keys
            else weights(false);
            tmem_store16(area, p);  // over the first half of the scores they came from
            asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            __syncwarp();
            if (lane == 0) mbar_arrive(p_full(tile & 1));
        }
        if (lane == 0) okay = mbar_wait(o_full, 0, abort_flag, t.spin_limit) && *abort_flag == 0;
        okay = __shfl_sync(0xffffffffu, okay ? 1 : 0, 0) != 0;
        if (okay) {
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            bf16* out = static_cast<bf16*>(a.out) + size_t(q0 + r) * a.out_pitch + size_t(head) * a.vdim;
            const bool there = q0 + r < a.tokens, wide = a.vdim % 8 == 0;  // (pitches are multiples of 64: rows of eight start at 16 bytes)
            for (int c = part * 16; c < a.vdim; c += 64) {
                uint32_t v[16];
                tmem_load16(mine + 2 * kLtKeys + c, v);
                asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
                if (!there) continue;
                if (wide) {
#pragma unroll
                    for (int i = 0; i < 2; ++i)
                        if (c + 8 * i < a.vdim)
                            *reinterpret_cast<uint4*>(out + c + 8 * i) =
                                make_uint4(pack_bf16(__uint_as_float(v[8 * i]), __uint_as_float(v[8 * i + 1])), pack_bf16(__uint_as_float(v[8 * i + 2]), __uint_as_float(v[8 * i + 3])),
                                           pack_bf16(__uint_as_float(v[8 * i + 4]), __uint_as_float(v[8 * i + 5])), pack_bf16(__uint_as_float(v[8 * i + 6]), __uint_as_float(v[8 * i + 7])));
                } else {
#pragma unroll
                    for (int i = 0; i < 16; ++i)
                        if (c + i < a.vdim) out[c + i] = __float2bfloat16_rn(__uint_as_float(v[i]));
                }
            }
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (tid == 0 && *abort_flag) atomicExch(t.status, kGemmStatusTimeout);
    if (warp == 0) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512u) : "memory");
    }
}

}  // namespace qtb
