// Pieces shared by the tcgen05 GEMM kernels: mbarrier / TMA helpers (bulk_async.cuh), the
// shared-memory matrix descriptor for 128-byte-swizzled K-major tiles, fences, commit and the
// tensor-memory load used by the epilogues.
#pragma once
#include <cuda.h>

#include "bulk_async.cuh"   // mbarrier + tensor-map helpers

namespace tc {

using gemvq8::mbar_arrive;
using gemvq8::mbar_expect_tx;
using gemvq8::mbar_init;
using gemvq8::mbar_wait;
using gemvq8::mbar_wait_spin;
using gemvq8::smem_u32;
using gemvq8::tma_load_2d;
using gemvq8::tma_load_3d;

constexpr int TM = 128;          // tokens per tile (UMMA M)
constexpr int TK = 64;           // K per stage: 64 f16 = 128 bytes = one swizzle row
constexpr int kStages = 4;
constexpr int kThreadsTc = 192;  // 6 warps

// 64-bit shared-memory matrix descriptor, K-major operand, 128-byte swizzle:
// rows of 128 bytes, 8-row groups 1024 bytes apart (SBO), descriptor version 1 (sm_100).
__device__ __forceinline__ uint64_t umma_desc_sw128(const void* smem_ptr) {
    const uint32_t addr = smem_u32(smem_ptr);
    uint64_t d = 0;
    d |= (uint64_t)((addr & 0x3FFFF) >> 4);            // start address, 16-byte units
    d |= (uint64_t)0 << 16;                            // leading byte offset: unused for swizzled K-major
    d |= (uint64_t)(1024 >> 4) << 32;                  // stride byte offset between 8-row groups
    d |= (uint64_t)1 << 46;                            // descriptor version
    d |= (uint64_t)2 << 61;                            // SWIZZLE_128B
    return d;
}

// 32-bit instruction descriptor, kind::f16: A and B both f16 or both bf16 (both K-major), f32 D, M x N tile.
__host__ __device__ constexpr uint32_t umma_idesc_f16(int m, int n, bool bf16 = false) {
    return (1u << 4)                      // D format f32
           | ((bf16 ? 1u : 0u) << 7) | ((bf16 ? 1u : 0u) << 10)   // A, B format: 0 = f16, 1 = bf16
           | (0u << 15) | (0u << 16)      // A, B K-major
           | ((uint32_t)(n >> 3) << 17) | ((uint32_t)(m >> 4) << 24);
}

__device__ __forceinline__ void tc_fence_after() { asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory"); }
__device__ __forceinline__ void tc_fence_before() { asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory"); }

__device__ __forceinline__ void umma_f16(uint32_t tmem_d, uint64_t adesc, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n\t.reg .pred p;\n\t"
        "setp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
        ::"r"(tmem_d), "l"(adesc), "l"(bdesc), "r"(idesc), "r"(accumulate)
        : "memory");
}
// arrive on `bar` once every tcgen05.mma issued so far by this thread has finished
__device__ __forceinline__ void umma_commit(uint64_t* bar) {
    asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(smem_u32(bar)) : "memory");
}
// 32 lanes x 32 consecutive f32 columns of tensor memory -> 32 registers per thread
__device__ __forceinline__ void tmem_ld_32x32(uint32_t taddr, float* v) {
    uint32_t r[32];
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x32.b32 "
        "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, "
        "%16, %17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31}, [%32];"
        : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]),
          "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]), "=r"(r[17]), "=r"(r[18]),
          "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]),
          "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
        : "r"(taddr)
        : "memory");
    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
    for (int i = 0; i < 32; ++i) v[i] = __uint_as_float(r[i]);
}

// 32 registers per thread -> 32 lanes x 32 columns of tensor memory
__device__ __forceinline__ void tmem_st_32x32(uint32_t taddr, const uint32_t* r) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
        "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, "
        "%17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};" ::"r"(taddr),
        "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]),
        "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(r[16]), "r"(r[17]), "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]),
        "r"(r[23]), "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31])
        : "memory");
    asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
}
// 32 lanes x 64 consecutive f32 columns of tensor memory -> 64 registers per thread
__device__ __forceinline__ void tmem_ld_32x64(uint32_t taddr, float* v) {
    uint32_t r[64];
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x64.b32 {"
        "%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, "
        "%16, %17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, "
        "%32, %33, %34, %35, %36, %37, %38, %39, %40, %41, %42, %43, %44, %45, %46, %47, "
        "%48, %49, %50, %51, %52, %53, %54, %55, %56, %57, %58, %59, %60, %61, %62, %63}, [%64];\n\t"
        "tcgen05.wait::ld.sync.aligned;"
        : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]),
          "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]),
          "=r"(r[16]), "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]), "=r"(r[23]),
          "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31]),
          "=r"(r[32]), "=r"(r[33]), "=r"(r[34]), "=r"(r[35]), "=r"(r[36]), "=r"(r[37]), "=r"(r[38]), "=r"(r[39]),
          "=r"(r[40]), "=r"(r[41]), "=r"(r[42]), "=r"(r[43]), "=r"(r[44]), "=r"(r[45]), "=r"(r[46]), "=r"(r[47]),
          "=r"(r[48]), "=r"(r[49]), "=r"(r[50]), "=r"(r[51]), "=r"(r[52]), "=r"(r[53]), "=r"(r[54]), "=r"(r[55]),
          "=r"(r[56]), "=r"(r[57]), "=r"(r[58]), "=r"(r[59]), "=r"(r[60]), "=r"(r[61]), "=r"(r[62]), "=r"(r[63])
        : "r"(taddr)
        : "memory");
#pragma unroll
    for (int i = 0; i < 64; ++i) v[i] = __uint_as_float(r[i]);
}
// 64 registers per thread -> 32 lanes x 64 columns of tensor memory
__device__ __forceinline__ void tmem_st_32x64(uint32_t taddr, const uint32_t* r) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x64.b32 [%0], {"
        "%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, "
        "%17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32, "
        "%33, %34, %35, %36, %37, %38, %39, %40, %41, %42, %43, %44, %45, %46, %47, %48, "
        "%49, %50, %51, %52, %53, %54, %55, %56, %57, %58, %59, %60, %61, %62, %63, %64};\n\t"
        "tcgen05.wait::st.sync.aligned;" ::"r"(taddr),
        "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]),
        "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]),
        "r"(r[16]), "r"(r[17]), "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]),
        "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31]),
        "r"(r[32]), "r"(r[33]), "r"(r[34]), "r"(r[35]), "r"(r[36]), "r"(r[37]), "r"(r[38]), "r"(r[39]),
        "r"(r[40]), "r"(r[41]), "r"(r[42]), "r"(r[43]), "r"(r[44]), "r"(r[45]), "r"(r[46]), "r"(r[47]),
        "r"(r[48]), "r"(r[49]), "r"(r[50]), "r"(r[51]), "r"(r[52]), "r"(r[53]), "r"(r[54]), "r"(r[55]),
        "r"(r[56]), "r"(r[57]), "r"(r[58]), "r"(r[59]), "r"(r[60]), "r"(r[61]), "r"(r[62]), "r"(r[63])
        : "memory");
}
// The same product with the A operand in tensor memory (a row per lane, two 16-bit elements of K per column)
__device__ __forceinline__ void umma_f16_ta(uint32_t tmem_d, uint32_t tmem_a, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n\t.reg .pred p;\n\t"
        "setp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}"
        ::"r"(tmem_d), "r"(tmem_a), "l"(bdesc), "r"(idesc), "r"(accumulate)
        : "memory");
}
// One lane of a converged warp.  A branch on it keeps the warp uniform for the compiler: the operands of the tensor-core instructions
// behind it go straight into uniform registers (behind `lane == 0` every instruction pays for moving them there: 140 to 190 cycles
// per tcgen05.mma were measured).
__device__ __forceinline__ bool elect_one() {
    uint32_t pred;
    asm volatile("{\n\t.reg .pred p;\n\telect.sync _|p, 0xffffffff;\n\tselp.u32 %0, 1, 0, p;\n\t}" : "=r"(pred));
    return pred != 0;
}
// Descriptor of a 128-byte-swizzled operand stored with its M / N dimension contiguous: 64 elements per 128-byte line, one line
// per k, 8-line groups 1024 bytes apart (SBO), 64-element blocks `block_bytes` apart (LBO).  The instruction descriptor then
// has the operand's transpose bit set (bit 16 for B).
__device__ __forceinline__ uint64_t umma_desc_sw128_mn(const void* smem_ptr, uint32_t block_bytes) {
    const uint32_t addr = smem_u32(smem_ptr);
    return (uint64_t)((addr & 0x3FFFF) >> 4) | (uint64_t)(block_bytes >> 4) << 16 | (uint64_t)(1024 >> 4) << 32 | (uint64_t)1 << 46 | (uint64_t)2 << 61;
}

// One 32 x 32 piece of an accumulator on its way to memory: a lane holds a row; turned around in shared memory, eight lanes handle 32
// consecutive columns of a row (four rows per pass), because rows are kilobytes apart and a lane per row writes 128-byte lines in
// sixteen-byte pieces (0.5 TB/s measured).  put(i, row of the piece, four values of this lane's columns 4 (lane % 8)..).
// `turn`: 256 float4s of the warp's own, places swizzled against bank conflicts.
constexpr int kTurnQuads = 32 * 8;
template <class Put> __device__ __forceinline__ void turn_piece(float4* turn, const float* v, Put put) {
    const int lane = threadIdx.x & 31, r = lane >> 3, quad = lane & 7;
#pragma unroll
    for (int j = 0; j < 8; ++j) turn[lane * 8 + (j ^ (lane & 7))] = make_float4(v[4 * j], v[4 * j + 1], v[4 * j + 2], v[4 * j + 3]);
    __syncwarp();
#pragma unroll
    for (int i = 0; i < 8; ++i) put(i, 4 * i + r, turn[(4 * i + r) * 8 + (quad ^ ((4 * i + r) & 7))]);
    __syncwarp();
}

// What the epilogue of a tensor-core GEMM does with an accumulator: Out = f16 / bf16: round(acc + bias);
// Out = f32: residual + alpha * (acc + bias), the residual stream of a model that keeps it in 32 bits
// (`resid` may be the output itself: every element is read by the thread that writes it).
template <class Out> struct GemmEpilogue {
    const Out* bias;          // per output column, nullable
    const float* resid;       // f32 output only, nullable
    float alpha;
    LinearAct act;            // after the bias
    __device__ __forceinline__ float value(float acc, int col) const {
        const float v = acc + (bias ? to_f32<Out>(bias[col]) : 0.f);
        return col < act.cols ? act(v) : v;
    }
    __device__ __forceinline__ Out operator()(float acc, int col, size_t idx) const {
        float v = value(acc, col);
        if (sizeof(Out) == 4) v = resid ? fmaf(alpha, v, resid[idx]) : alpha * v;
        return from_f32<Out>(v);
    }
    // four consecutive columns whose bias, and residual (f32 output), the caller has loaded; `col` a multiple of 4
    struct alignas(4 * sizeof(Out)) Quad { Out v[4]; };
    __device__ __forceinline__ float4 bias4(int col) const {
        return bias ? make_float4(to_f32<Out>(bias[col]), to_f32<Out>(bias[col + 1]), to_f32<Out>(bias[col + 2]), to_f32<Out>(bias[col + 3])) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    __device__ __forceinline__ void store4(Out* out, size_t idx, const float4& acc, const float4& b, const float4& r, int col) const {
        float v[4] = {acc.x + b.x, acc.y + b.y, acc.z + b.z, acc.w + b.w};
        if (col < act.cols) {
            if (act.kind == RCU_ACT_RELU_SQUARED) {      // without branches: the others are dear enough to hide them
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float p = fmaxf(v[e], 0.f);
                    v[e] = col + e < act.cols ? p * p : v[e];
                }
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e) v[e] = col + e < act.cols ? act(v[e]) : v[e];
            }
        }
        if (sizeof(Out) == 4) {
            v[0] = resid ? fmaf(alpha, v[0], r.x) : alpha * v[0];
            v[1] = resid ? fmaf(alpha, v[1], r.y) : alpha * v[1];
            v[2] = resid ? fmaf(alpha, v[2], r.z) : alpha * v[2];
            v[3] = resid ? fmaf(alpha, v[3], r.w) : alpha * v[3];
        }
        Quad q;
#pragma unroll
        for (int e = 0; e < 4; ++e) q.v[e] = from_f32<Out>(v[e]);
        *reinterpret_cast<Quad*>(out + idx) = q;
    }
    // eight consecutive columns, 16-byte aligned
    __device__ __forceinline__ void store8(Out* out, size_t idx, const float* acc, int col) const {
        __align__(16) Out h[8];
        if (sizeof(Out) == 4 && resid) {
            __align__(16) float r[8];
            *reinterpret_cast<float4*>(r) = *reinterpret_cast<const float4*>(resid + idx);
            *reinterpret_cast<float4*>(r + 4) = *reinterpret_cast<const float4*>(resid + idx + 4);
#pragma unroll
            for (int e = 0; e < 8; ++e) h[e] = from_f32<Out>(fmaf(alpha, value(acc[e], col + e), r[e]));
        } else {
#pragma unroll
            for (int e = 0; e < 8; ++e) h[e] = (*this)(acc[e], col + e, idx + e);
        }
#pragma unroll
        for (int v = 0; v < (int)sizeof(Out) / 2; ++v) reinterpret_cast<uint4*>(out + idx)[v] = reinterpret_cast<const uint4*>(h)[v];
    }
};

}  // namespace tc

// Host-side description of a 16-bit tensor-core Linear beyond its sizes (rcu_linear): operand type, row pitch of the
// activations in elements (0: K), output type and the f32 epilogue.
struct TcLinear {
    bool bf16 = false;
    uint64_t x_pitch = 0;
    int out_dt = RCU_F16;
    const float* resid = nullptr;
    float alpha = 1.f;
    LinearAct act = {};
};
