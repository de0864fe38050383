// Masked attention of a long bf16 block on the 5th-generation tensor cores (tcgen05), behind the interfaces of
// rcu_window_attention and rcu_grouped_attention (rcu_attend in latent_attention.cu sends blocks of at least 256 tokens here).
//
// CTA = 256 queries of one head, in two tiles of 128 that take turns: while the softmax warps of one tile work, the tensor core
// runs the other tile's products.
//   warp 0 (one lane)   TMA producer: the queries once, then 64 keys (own and shared features) and their values per stage;
//   warp 1              per key tile n and query tile w: S_w = Q_w K^T into tensor memory, then O_w += P_w V of tile n - 1 with
//                       P_w read from tensor memory - its value and its remainder, two products, so that attention weights
//                       keep 16 bits of mantissa.  S and P of consecutive key tiles have buffers of their own, so the scores of a
//                       tile are there before the weights of the one before are;
//   warps 2-5, 6-9      softmax of tile 0 / 1, a query per thread: scores from tensor memory, mask, running maximum, weights
//                       back over the scores.  The maximum that weights are taken against only moves when a score exceeds it
//                       by more than 2^8, so that O_w is rescaled rarely; all of it is f32.
// Tensor memory per query tile: two buffers of 64 columns (S, then P), up to 128 columns O.  A query tile passes over key tiles none
// of its queries sees.  CTAs with many key tiles start first.  Every wait is bounded; one that gives up raises RCU_DEVFLAG_TIMEOUT and
// ends all others of the CTA.
#include <cuda.h>

#include "lm_mma.cuh"
#include "tc_common.cuh"
#include "window.cuh"

namespace {

using namespace tc;

constexpr int kTileQ = 128, kTileK = 64, kThreadsW = 320;
constexpr int kBlockQ = kTileQ * 128, kBlockK = kTileK * 128;       // bytes of 64 columns of a query / key tile

struct TcArgs {
    __nv_bfloat16* out;
    int T, L, H, G, D, R, E;
    Visible see;
    float scale;
    const float* sink;
    int* status;
};

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// The i-th query block to start of n: blocks late in a chunk (without chunks: late in the sequence) see the most keys and go first.
__device__ __forceinline__ int heavy_first(int i, int n, int chunk) {
    const int p = chunk > 0 ? min(n, max(1, (chunk + kTileQ) / (2 * kTileQ))) : n;        // blocks per chunk
    const int full = n / p, more = n - full * p, head = (p - more) * full;               // `more` places of a chunk occur once more than the others
    if (i < head) return i % full * p + p - 1 - i / full;
    i -= head;
    return i % (full + 1) * p + more - 1 - i / (full + 1);
}

// NB: 64-column blocks of a query (own features, then shared ones; columns beyond the features are zero)
template <int NB>
__global__ void __launch_bounds__(kThreadsW, 1)
window_tc_kernel(const __grid_constant__ CUtensorMap qmap, const __grid_constant__ CUtensorMap qrmap, const __grid_constant__ CUtensorMap kmap,
                 const __grid_constant__ CUtensorMap krmap, const __grid_constant__ CUtensorMap vmap, const TcArgs a) {
    rcu_kernel_entry_wait_only();
    extern __shared__ unsigned char smem_dyn[];
    constexpr int nb = NB;
    const int nd = (a.D + 63) / 64, eb = (a.E + 63) / 64;      // 64-column blocks
    unsigned char* qs = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_dyn) + 1023) & ~(uintptr_t)1023);
    unsigned char* ks = qs + 2 * nb * kBlockQ;
    unsigned char* vs = ks + 2 * nb * kBlockK;
    __shared__ __align__(8) uint64_t q_full, k_full[2], k_empty[2], v_full[2], v_empty[2], s_full[2][2], p_full[2][2], pv_done[2], drained;
    __shared__ uint32_t tmem_slot;
    __shared__ volatile int abort_flag;

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int h = blockIdx.x, hk = h / (a.H / a.G), i0 = heavy_first(blockIdx.y, gridDim.y, a.see.chunk) * 2 * kTileQ;
    const int base = a.L - a.T + i0, nq = min(2 * kTileQ, a.T - i0);    // key row of the CTA's first query; its queries
    const int first = a.see.first(base);
    const int tiles = (base + nq - 1 - first) / kTileK + 1;
    // key tiles [lo, hi) that some query of tile w sees
    auto lo_of = [&](int w) { return (a.see.first(base + w * kTileQ) - first) / kTileK; };
    auto hi_of = [&](int w) { return w * kTileQ < nq ? (min(base + (w + 1) * kTileQ, base + nq) - 1 - first) / kTileK + 1 : 0; };

    if (threadIdx.x == 0) {
        mbar_init(&q_full, 1);
        mbar_init(&drained, 1);
        for (int i = 0; i < 2; ++i) {
            mbar_init(&k_full[i], 1);
            mbar_init(&k_empty[i], 1);
            mbar_init(&v_full[i], 1);
            mbar_init(&v_empty[i], 1);
            for (int b = 0; b < 2; ++b) {
                mbar_init(&s_full[i][b], 1);
                mbar_init(&p_full[i][b], 4);
            }
            mbar_init(&pv_done[i], 1);
        }
        abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_slot)), "n"(512) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_slot;

    if (warp == 0) {
        if (lane == 0) {
            mbar_expect_tx(&q_full, 2 * nb * kBlockQ);
            for (int w = 0; w < 2; ++w)
                for (int b = 0; b < nb; ++b)
                    tma_load_3d(qs + (w * nb + b) * kBlockQ, b < nd ? &qmap : &qrmap, (b < nd ? b : b - nd) * 64, h, i0 + w * kTileQ, &q_full);
            // keys run one tile ahead of values
            for (int n = 0; n <= tiles; ++n) {
                if (n < tiles) {
                    const int s = n & 1, j0 = first + n * kTileK;
                    if (n >= 2 && !mbar_wait(&k_empty[s], ((n >> 1) - 1) & 1, &abort_flag, a.status)) break;
                    mbar_expect_tx(&k_full[s], nb * kBlockK);
                    for (int b = 0; b < nd; ++b) tma_load_3d(ks + (s * nb + b) * kBlockK, &kmap, b * 64, hk, j0, &k_full[s]);
                    for (int b = nd; b < nb; ++b) tma_load_2d(ks + (s * nb + b) * kBlockK, &krmap, (b - nd) * 64, j0, &k_full[s]);
                }
                if (n > 0) {
                    const int v = n - 1, s = v & 1, j0 = first + v * kTileK;
                    if (v >= 2 && !mbar_wait(&v_empty[s], ((v >> 1) - 1) & 1, &abort_flag, a.status)) break;
                    mbar_expect_tx(&v_full[s], eb * kBlockK);
                    for (int b = 0; b < eb; ++b) tma_load_3d(vs + (s * eb + b) * kBlockK, &vmap, b * 64, hk, j0, &v_full[s]);
                }
            }
        }
    } else if (warp == 1) {
        // the whole warp keeps step, one elected lane issues
        const uint32_t idesc_s = umma_idesc_f16(kTileQ, kTileK, true);
        const uint32_t idesc_o = umma_idesc_f16(kTileQ, (a.E + 15) & ~15, true) | (1u << 16);     // V is stored with its columns contiguous
        const int lo[2] = {lo_of(0), lo_of(1)}, hi[2] = {hi_of(0), hi_of(1)};
        const uint64_t qd = umma_desc_sw128(qs), kd = umma_desc_sw128(ks), vd = umma_desc_sw128_mn(vs, kBlockK);
        const bool leader = elect_one();
        auto wait = [&](uint64_t* bar, int phase) { return (bool)__all_sync(0xffffffffu, mbar_wait_spin(bar, phase & 1, &abort_flag, a.status)); };
        bool ok = wait(&q_full, 0);
        tc_fence_after();
        for (int n = 0; n <= tiles && ok; ++n) {
            const int s = n & 1, p = s ^ 1;
            if (n < tiles) {
                ok = wait(&k_full[s], n >> 1);
#pragma unroll
                for (int w = 0; w < 2; ++w) {
                    if (!ok || n < lo[w] || n >= hi[w]) continue;
                    // the buffer's last weights have been read
                    if (n - 2 >= lo[w]) ok = wait(&pv_done[w], n - 2 - lo[w]);
                    if (!ok) continue;
                    tc_fence_after();
                    if (leader) {
                        const uint32_t t = tmem + (uint32_t)w * 256 + 64 * s;
                        const uint64_t bd = kd + (uint64_t)(s * NB * (kBlockK >> 4));
#pragma unroll
                        for (int b = 0; b < NB; ++b)
#pragma unroll
                            for (int k = 0; k < 4; ++k)
                                umma_f16(t, qd + (w * NB + b) * (kBlockQ >> 4) + 2 * k, bd + b * (kBlockK >> 4) + 2 * k, idesc_s, (b > 0 || k > 0) ? 1u : 0u);
                        umma_commit(&s_full[w][s]);
                    }
                    __syncwarp();
                }
                if (!ok) break;
                if (leader) umma_commit(&k_empty[s]);
                __syncwarp();
            }
            if (n > 0) {
                ok = wait(&v_full[p], (n - 1) >> 1);
#pragma unroll
                for (int w = 0; w < 2; ++w) {
                    if (!ok || n - 1 < lo[w] || n - 1 >= hi[w]) continue;
                    ok = wait(&p_full[w][p], (n - 1 - lo[w]) >> 1);
                    if (!ok) continue;
                    tc_fence_after();
                    if (leader) {
                        const uint32_t t = tmem + (uint32_t)w * 256;
                        const uint64_t bd = vd + (uint64_t)(p * eb * (kBlockK >> 4));
                        const uint32_t more = n - 1 > lo[w] ? 1u : 0u;
#pragma unroll
                        for (int half = 0; half < 2; ++half)          // weights, then their remainders
#pragma unroll
                            for (int k = 0; k < kTileK / 16; ++k)      // 16 keys are two 1024-byte groups of V, eight columns of P
                                umma_f16_ta(t + 128, t + 64 * p + 32 * half + 8 * k, bd + 128 * k, idesc_o, half > 0 || k > 0 ? 1u : more);
                        umma_commit(&pv_done[w]);
                    }
                    __syncwarp();
                }
                if (!ok) break;
                if (leader) umma_commit(&v_empty[p]);
                __syncwarp();
            }
        }
        if (!ok && leader) {            // given up: let the products in flight end before tensor memory is freed
            umma_commit(&drained);
            for (int i = 0; i < (1 << 20) && !gemvq8::mbar_test_wait(&drained, 0); ++i) {}
        }
        __syncwarp();
    } else {
        const int w = warp < 6 ? 0 : 1, quarter = warp & 3;
        const int r = w * kTileQ + quarter * 32 + lane, row = base + r;        // query of the CTA, its key row
        const int lo = lo_of(w), hi = hi_of(w);
        const uint32_t t = tmem + (uint32_t)w * 256 + ((uint32_t)(quarter * 32) << 16);
        const int row0 = base + w * kTileQ + quarter * 32, row1 = row0 + 31;   // the warp's key rows
        const int low = a.see.first(row), low1 = a.see.first(row1);
        const float sc = a.scale * 1.4426950408889634f;                       // scores in units of log 2
        const int ocols = (a.E + 31) & ~31;
        float m = -INFINITY, l = 0.f;
        bool ok = true;
        for (int n = lo; n < hi; ++n) {
            const int b = n & 1;
            ok = __all_sync(0xffffffffu, mbar_wait_spin(&s_full[w][b], ((n - lo) >> 1) & 1, &abort_flag, a.status));
            if (!ok) break;
            tc_fence_after();
            float s[64];
            tmem_ld_32x64(t + 64 * b, s);
            const int j0 = first + n * kTileK;
            if (j0 + kTileK - 1 > row0 || j0 < low1) {
#pragma unroll
                for (int j = 0; j < 64; ++j)
                    if (j0 + j > row || j0 + j < low) s[j] = -INFINITY;
            }
            float top4[4] = {s[0], s[1], s[2], s[3]};
#pragma unroll
            for (int j = 4; j < 64; ++j) top4[j & 3] = fmaxf(top4[j & 3], s[j]);
            const float top = fmaxf(fmaxf(top4[0], top4[1]), fmaxf(top4[2], top4[3])) * sc;      // sc > 0
            const bool move = top > m + 8.f || (m == -INFINITY && top > -INFINITY);
            const float next = move ? top : m;
            const float corr = move ? ex2(m - next) : 1.f;                    // 0 while no key has been seen
            m = next;
            const float z = m == -INFINITY ? 0.f : -m;
            float l4[4] = {l * corr, 0.f, 0.f, 0.f};
            uint32_t pw[64];                                                  // weights, then their remainders
#pragma unroll
            for (int j = 0; j < 32; ++j) {
                const float x = ex2(fmaf(s[2 * j], sc, z)), y = ex2(fmaf(s[2 * j + 1], sc, z));
                l4[j & 3] += x + y;
                lm::split2(x, y, pw[j], pw[32 + j]);
            }
            l = (l4[0] + l4[1]) + (l4[2] + l4[3]);
            // O may be rescaled once the product of the tile before has been added.  The last tile always waits for that: a wait for
            // the last product then never looks two completions back.
            const bool any = __any_sync(0xffffffffu, move);
            if (n > lo && (any || n == hi - 1)) {
                ok = __all_sync(0xffffffffu, mbar_wait_spin(&pv_done[w], (n - lo - 1) & 1, &abort_flag, a.status));
                if (!ok) break;
                tc_fence_after();
                if (any) {
                    for (int c = 0; c < ocols; c += 32) {
                        float o[32];
                        tmem_ld_32x32(t + 128 + c, o);
#pragma unroll
                        for (int j = 0; j < 32; ++j) o[j] *= corr;
                        tmem_st_32x32(t + 128 + c, reinterpret_cast<const uint32_t*>(o));
                    }
                }
            }
            tmem_st_32x64(t + 64 * b, pw);
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&p_full[w][b]);
        }
        if (ok && hi > lo) {
            ok = __all_sync(0xffffffffu, mbar_wait(&pv_done[w], (hi - lo - 1) & 1, &abort_flag, a.status));
            tc_fence_after();
            if (ok) {
                if (a.sink) l += ex2(a.sink[h] * 1.4426950408889634f - m);
                const float inv = 1.0f / l;
                __nv_bfloat16* out = a.out + ((size_t)(i0 + r) * a.H + h) * a.E;
                for (int c = 0; c < ocols; c += 32) {
                    float o[32];
                    tmem_ld_32x32(t + 128 + c, o);
                    if (r < nq) {
#pragma unroll
                        for (int j = 0; j < 32; j += 8)
                            if (c + j < a.E) {          // E is a multiple of 8
                                __align__(16) __nv_bfloat16 v[8];
#pragma unroll
                                for (int e = 0; e < 8; ++e) v[e] = __float2bfloat16_rn(o[j + e] * inv);
                                *reinterpret_cast<uint4*>(out + c + j) = *reinterpret_cast<const uint4*>(v);
                            }
                    }
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "n"(512) : "memory");
    }
}

// [cols of a head, heads, rows] bf16, a box of 64 columns x `rows` rows of one head, 128-byte swizzle; columns beyond the head's are zero
bool make_head_map(CUtensorMap* map, const void* base, uint64_t cols, uint64_t heads, uint64_t rows, uint64_t head_pitch, uint64_t row_pitch, uint32_t box_rows) {
    gemvq8::EncodeTiledFn fn = gemvq8::encode_tiled_fn();
    if (!fn) return false;
    cuuint64_t dims[3] = {cols, heads, rows};
    cuuint64_t strides[2] = {head_pitch * 2, row_pitch * 2};
    cuuint32_t box[3] = {64, 1, box_rows};
    cuuint32_t estr[3] = {1, 1, 1};
    return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
              CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}
bool make_row_map(CUtensorMap* map, const void* base, uint64_t cols, uint64_t rows, uint64_t pitch, uint32_t box_rows) {
    gemvq8::EncodeTiledFn fn = gemvq8::encode_tiled_fn();
    if (!fn) return false;
    cuuint64_t dims[2] = {cols, rows};
    cuuint64_t strides[1] = {pitch * 2};
    cuuint32_t box[2] = {64, box_rows};
    cuuint32_t estr[2] = {1, 1};
    return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
              CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

}  // namespace

rcu_status rcu_window_tc(rcu_device* dev, const WindowArgs& a) {
    const int Q = a.D + a.R, nb = (a.D + 63) / 64 + (a.R + 63) / 64, eb = (a.E + 63) / 64;
    if (!(a.scale > 0.f) || a.T < 256 || a.T > 65535 * 2 * kTileQ || a.D < 8 || a.D % 8 || a.R % 8 || a.E % 8 || a.E > 128 || nb > 4 || a.shared_pitch % 8) return RCU_ERR_UNSUPPORTED;
    if ((reinterpret_cast<uintptr_t>(a.q) | reinterpret_cast<uintptr_t>(a.kv) | reinterpret_cast<uintptr_t>(a.shared) | reinterpret_cast<uintptr_t>(a.out)) & 15)
        return RCU_ERR_UNSUPPORTED;
    const size_t smem = 1024 + (size_t)2 * nb * kBlockQ + (size_t)2 * (nb + eb) * kBlockK;
    if (smem + 512 > (size_t)dev->smem_optin) return RCU_ERR_UNSUPPORTED;
    const __nv_bfloat16 *q = (const __nv_bfloat16*)a.q, *kv = (const __nv_bfloat16*)a.kv;
    const uint64_t kvp = (uint64_t)a.G * (a.D + a.E), qp = (uint64_t)a.H * Q;
    CUtensorMap qm, qr, km, kr, vm;
    if (!make_head_map(&qm, q, a.D, a.H, a.T, Q, qp, kTileQ) || !make_head_map(&km, kv, a.D, a.G, a.L, a.D, kvp, kTileK) ||
        !make_head_map(&vm, kv + (size_t)a.G * a.D, a.E, a.G, a.L, a.E, kvp, kTileK))
        return rcu_fail(dev, RCU_ERR_CUDA, "window_attention: cuTensorMapEncodeTiled failed (T=%d L=%d H=%d)", a.T, a.L, a.H);
    if (a.R == 0) {
        qr = qm;              // no shared features: never read
        kr = km;
    } else if (!make_head_map(&qr, q + a.D, a.R, a.H, a.T, Q, qp, kTileQ) || !make_row_map(&kr, a.shared, a.R, a.L, a.shared_pitch, kTileK))
        return rcu_fail(dev, RCU_ERR_CUDA, "window_attention: cuTensorMapEncodeTiled failed (T=%d L=%d H=%d)", a.T, a.L, a.H);
    const TcArgs t{(__nv_bfloat16*)a.out, a.T, a.L, a.H, a.G, a.D, a.R, a.E, a.see, a.scale, a.sink, dev->d_status};
    const dim3 grid(a.H, (a.T + 2 * kTileQ - 1) / (2 * kTileQ));
    void (*kern)(CUtensorMap, CUtensorMap, CUtensorMap, CUtensorMap, CUtensorMap, TcArgs) =
        nb == 1 ? window_tc_kernel<1> : nb == 2 ? window_tc_kernel<2> : nb == 3 ? window_tc_kernel<3> : window_tc_kernel<4>;
    RCU_CUDA(dev, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    RCU_CUDA(dev, rcu_launch(dev, kern, grid, kThreadsW, smem, qm, qr, km, kr, vm, t));
    RCU_LAUNCH_CHECK(dev);
    return RCU_OK;
}
