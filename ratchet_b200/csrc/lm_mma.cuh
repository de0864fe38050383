// Warp-level bf16 tensor-core pieces of the chunked linear attention and the windowed attention: ldmatrix operand loads,
// mma.sync m16n8k16 with f32 accumulation, and the two-term bf16 form of an f32 operand (value and remainder: 16 bits of
// mantissa), which keeps attention weights and recurrent states at f32-like accuracy through a bf16 product.
#pragma once
#include "lm_math.cuh"

namespace lm {

using bf16 = __nv_bfloat16;

__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }

// A operand, 16 x 16 at rows r0.., columns k0.. of a row-major tile with `ld` elements per row
__device__ __forceinline__ void load_a(uint32_t (&a)[4], const bf16* tile, int ld, int r0, int k0) {
    const int lane = threadIdx.x & 31;
    const uint32_t p = smem_addr(tile + (size_t)(r0 + (lane & 15)) * ld + k0 + (lane >> 4) * 8);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(a[0]), "=r"(a[1]), "=r"(a[2]), "=r"(a[3]) : "r"(p));
}
// A operand from a tile stored transposed: element (row, k) at tile[k][row]
__device__ __forceinline__ void load_a_t(uint32_t (&a)[4], const bf16* tile, int ld, int r0, int k0) {
    const int lane = threadIdx.x & 31;
    const uint32_t p = smem_addr(tile + (size_t)(k0 + (lane & 7) + (lane >> 4) * 8) * ld + r0 + ((lane >> 3) & 1) * 8);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(a[0]), "=r"(a[1]), "=r"(a[2]), "=r"(a[3]) : "r"(p));
}
// B operands of two neighbouring 8-column tiles, 16 deep, from a tile stored [column][k] (b[0], b[1]: columns n0.., b[2], b[3]: n0 + 8..)
__device__ __forceinline__ void load_b(uint32_t (&b)[4], const bf16* tile, int ld, int n0, int k0) {
    const int lane = threadIdx.x & 31;
    const uint32_t p = smem_addr(tile + (size_t)(n0 + (lane & 7) + (lane >> 4) * 8) * ld + k0 + ((lane >> 3) & 1) * 8);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(b[0]), "=r"(b[1]), "=r"(b[2]), "=r"(b[3]) : "r"(p));
}
// the same from a tile stored [k][column]
__device__ __forceinline__ void load_b_t(uint32_t (&b)[4], const bf16* tile, int ld, int n0, int k0) {
    const int lane = threadIdx.x & 31;
    const uint32_t p = smem_addr(tile + (size_t)(k0 + (lane & 15)) * ld + n0 + (lane >> 4) * 8);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(b[0]), "=r"(b[1]), "=r"(b[2]), "=r"(b[3]) : "r"(p));
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

__device__ __forceinline__ uint32_t pack(bf16 lo, bf16 hi) {
    return (uint32_t)__bfloat16_as_ushort(lo) | ((uint32_t)__bfloat16_as_ushort(hi) << 16);
}
// two f32 values as packed bf16 pairs: their roundings and the roundings of what those left over
__device__ __forceinline__ void split2(float x, float y, uint32_t& value, uint32_t& rest) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(x, y);
    value = *reinterpret_cast<const uint32_t*>(&v);
    const __nv_bfloat162 r = __floats2bfloat162_rn(x - __uint_as_float(value << 16), y - __uint_as_float(value & 0xffff0000u));
    rest = *reinterpret_cast<const uint32_t*>(&r);
}

__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool valid) {
    const int bytes = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_addr(dst)), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// rows x cols elements of a row-major matrix (row `r` at src + r * pitch) into a tile with `ld` elements per row, `tile_cols` wide
// (a multiple of 8); rows from `valid_rows` on and columns from `cols` on become zero.  vec: every row starts on 16 bytes and cols
// is a multiple of 8 (asynchronous copies: commit and wait).
__device__ __forceinline__ void load_tile(bf16* tile, int ld, const bf16* src, long long pitch, int rows, int valid_rows, int cols, int tile_cols, bool vec) {
    const int per = tile_cols / 8;
    for (int i = threadIdx.x; i < rows * per; i += blockDim.x) {
        const int r = i / per, c = (i - r * per) * 8;
        bf16* dst = tile + (size_t)r * ld + c;
        const bf16* s = src + (long long)r * pitch + c;
        if (vec) {
            const bool ok = r < valid_rows && c < cols;
            cp_async16(dst, ok ? s : src, ok);
        } else {
            __align__(16) bf16 v[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) v[e] = r < valid_rows && c + e < cols ? s[e] : __float2bfloat16_rn(0.f);
            *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<const uint4*>(v);
        }
    }
}

}  // namespace lm
