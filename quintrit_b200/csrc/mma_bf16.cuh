// Warp-level bf16 products with 32-bit sums (mma.sync m16n8k16) for kernels whose operands come out of registers: chunked recurrences and
// attention of many tokens. A 32-bit operand goes in as two bf16 terms (hi + lo), which keeps about 16 bits of it.
#pragma once
#include "dense_gemv.cuh"

namespace qtb {

// D(16 x 8) += A(16 x 16) B(16 x 8). Lane (g = lane / 4, c = lane % 4) holds A rows g, g + 8 at columns 2c, 2c + 1 (a0, a1) and 2c + 8, 2c + 9
// (a2, a3), B rows 2c, 2c + 1 (b0) and 2c + 8, 2c + 9 (b1) of column g, D rows g (d0, d1) and g + 8 (d2, d3) at columns 2c, 2c + 1.
__device__ __forceinline__ void mma_16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(static_cast<uint32_t>(__cvta_generic_to_shared(p)))
                 : "memory");
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(static_cast<uint32_t>(__cvta_generic_to_shared(p)))
                 : "memory");
}
// Fragments of a 16 x 16 bf16 tile at `tile` (row pitch in elements, rows 16-byte aligned). Read as it lies it is an A operand (rows m, columns
// k); read transposed, with rows k and columns n, it is two B operands: r[0], r[1] for columns 0..7 and r[2], r[3] for 8..15.
__device__ __forceinline__ void load_frag_a(uint32_t (&r)[4], const bf16* tile, int pitch) {
    const int lane = threadIdx.x & 31;
    ldmatrix_x4(r, tile + size_t(lane & 15) * pitch + (lane >> 4) * 8);
}
__device__ __forceinline__ void load_frag_b(uint32_t (&r)[4], const bf16* tile, int pitch) {
    const int lane = threadIdx.x & 31;
    ldmatrix_x4_trans(r, tile + size_t(lane & 15) * pitch + (lane >> 4) * 8);
}
// Two B operands from a tile stored with rows n and columns k (keys of an attention): r[0], r[1] for rows 0..7 and r[2], r[3] for 8..15.
__device__ __forceinline__ void load_frag_bt(uint32_t (&r)[4], const bf16* tile, int pitch) {
    const int lane = threadIdx.x & 31;
    ldmatrix_x4(r, tile + size_t((lane & 7) + (lane >> 4) * 8) * pitch + ((lane >> 3) & 1) * 8);
}
__device__ __forceinline__ uint32_t pack_bf16(float x, float y) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(x, y);
    return *reinterpret_cast<const uint32_t*>(&v);
}
__device__ __forceinline__ void split_bf16(float x, float y, uint32_t* hi, uint32_t* lo) {
    *hi = pack_bf16(x, y);
    *lo = pack_bf16(x - __uint_as_float(*hi << 16), y - __uint_as_float(*hi & 0xffff0000u));
}
__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool valid) {  // zeros where not valid
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(dst))), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_commit_group() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait_group() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

}  // namespace qtb
