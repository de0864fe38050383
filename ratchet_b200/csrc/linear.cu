// Linear with a chosen output type: out[M, N] = x[M, K] . W[N, K]^T (+ bias), rounded to the operands' type or kept in
// f32 as resid + alpha * (...), with an activation on the leading columns.  It is what a model with a 32-bit residual stream and
// 16-bit projections needs beside
// rcu_matmul, whose output has the activations' type (ops/matmul/mod.rs:484-495).
//
//   16-bit operands, shapes the tensor maps take: the tcgen05 kernels of gemm_tc2.cu / gemm_tc.cu;
//   up to four token rows: one warp per weight row (the weights are read once, whatever the type);
//   everything else, and every f32 product: 64 x 64 tiles in f32 FFMA - an f32 model runs in true 32-bit.
#include "tc_common.cuh"

rcu_status rcu_gemm_tc_linear(rcu_device* dev, const void* w, const void* x, const void* bias, void* y, uint64_t M, uint64_t N, uint64_t K,
                              const TcLinear& t);

namespace {

using tc::GemmEpilogue;

constexpr int kSkinny = 4;       // token rows the warp-per-row kernel takes

template <class T, class Out>
__global__ void __launch_bounds__(256)
linear_skinny_kernel(const T* __restrict__ W, const T* __restrict__ x, long long x_pitch, const GemmEpilogue<Out> epi, Out* out, int M, int N, int K,
                     int aligned) {
    rcu_kernel_entry();
    constexpr int VEC = 16 / (int)sizeof(T);
    const int lane = threadIdx.x & 31;
    const int n = blockIdx.x * 8 + (threadIdx.x >> 5);
    if (n >= N) return;
    float acc[kSkinny] = {0.f, 0.f, 0.f, 0.f};
    const T* row = W + (size_t)n * K;
    if (aligned) {
#pragma unroll 4
        for (int k = lane * VEC; k < K; k += 32 * VEC) {
            const uint4 wv = ld_stream_v4(row + k);
            const T* wt = reinterpret_cast<const T*>(&wv);
#pragma unroll
            for (int m = 0; m < kSkinny; ++m) {
                if (m >= M) break;
                const uint4 xv = *reinterpret_cast<const uint4*>(x + m * x_pitch + k);
                const T* xt = reinterpret_cast<const T*>(&xv);
#pragma unroll
                for (int e = 0; e < VEC; ++e) acc[m] = fmaf(to_f32<T>(wt[e]), to_f32<T>(xt[e]), acc[m]);
            }
        }
    } else {
        for (int k = lane; k < K; k += 32) {
            const float wf = to_f32<T>(row[k]);
#pragma unroll
            for (int m = 0; m < kSkinny; ++m)
                if (m < M) acc[m] = fmaf(wf, to_f32<T>(x[m * x_pitch + k]), acc[m]);
        }
    }
#pragma unroll
    for (int m = 0; m < kSkinny; ++m) acc[m] = warp_sum(acc[m]);
    if (lane == 0)
        for (int m = 0; m < M; ++m) out[(size_t)m * N + n] = epi(acc[m], n, (size_t)m * N + n);
}

constexpr int BM = 64, BN = 64, BK = 16;

template <class T, class Out>
__global__ void __launch_bounds__(256)
linear_simt_kernel(const T* __restrict__ W, const T* __restrict__ x, long long x_pitch, const GemmEpilogue<Out> epi, Out* out, int M, int N, int K) {
    rcu_kernel_entry();
    __shared__ float Xs[BK][BM + 4];
    __shared__ float Ws[BK][BN + 4];
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int m0 = blockIdx.y * BM, n0 = blockIdx.x * BN;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < K; k0 += BK) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int idx = tid + e * 256, k = idx % BK, i = idx / BK;
            const bool kk = k0 + k < K;
            Xs[k][i] = (kk && m0 + i < M) ? to_f32<T>(x[(long long)(m0 + i) * x_pitch + k0 + k]) : 0.f;
            Ws[k][i] = (kk && n0 + i < N) ? to_f32<T>(W[(size_t)(n0 + i) * K + k0 + k]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < BK; ++k) {
            const float4 a = *reinterpret_cast<const float4*>(&Xs[k][ty * 4]);
            const float4 b = *reinterpret_cast<const float4*>(&Ws[k][tx * 4]);
            const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int m = m0 + ty * 4 + i;
        if (m >= M) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int n = n0 + tx * 4 + j;
            if (n < N) out[(size_t)m * N + n] = epi(acc[i][j], n, (size_t)m * N + n);
        }
    }
}

template <class T, class Out>
rcu_status launch_plain(rcu_device* dev, const void* w, const void* x, uint64_t pitch, const void* bias, const float* resid, float alpha, const LinearAct& act, void* y,
                        uint64_t M, uint64_t N, uint64_t K) {
    const GemmEpilogue<Out> epi{(const Out*)bias, resid, alpha, act};
    if (M <= (uint64_t)kSkinny) {
        constexpr uint64_t VEC = 16 / sizeof(T);
        const int aligned = K % VEC == 0 && pitch % VEC == 0 && ((reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(x)) & 15) == 0;
        rcu_launch(dev, linear_skinny_kernel<T, Out>, (unsigned)((N + 7) / 8), 256, 0, (const T*)w, (const T*)x, (long long)pitch, epi, (Out*)y, (int)M,
                   (int)N, (int)K, aligned);
    } else {
        const dim3 grid((unsigned)((N + BN - 1) / BN), (unsigned)((M + BM - 1) / BM));
        RCU_REQUIRE(dev, grid.y <= 65535, "linear: too many token rows for the SIMT kernel");
        rcu_launch(dev, linear_simt_kernel<T, Out>, grid, 256, 0, (const T*)w, (const T*)x, (long long)pitch, epi, (Out*)y, (int)M, (int)N, (int)K);
    }
    RCU_LAUNCH_CHECK(dev);
    return RCU_OK;
}

}  // namespace

extern "C" rcu_status rcu_linear(rcu_device* dev, const rcu_tensor* w, const rcu_tensor* x, uint32_t x_col, const rcu_tensor* bias,
                                 int act, uint32_t act_cols, float act_param, const rcu_tensor* resid, float alpha, rcu_tensor* dst) {
    if (!dev) return RCU_ERR_INVALID_ARG;
    RCU_REQUIRE(dev, t_valid(w) && t_valid(x) && t_valid(dst), "linear: invalid tensor descriptor");
    RCU_REQUIRE(dev, w->rank == 2 && w->dt == x->dt && dt_is_float(w->dt), "linear: w must be a float matrix of the activations' dtype");
    RCU_REQUIRE(dev, dst->dt == x->dt || dst->dt == RCU_F32, "linear: the output is f32 or has the activations' dtype");
    const uint64_t N = w->shape[0], K = w->shape[1], pitch = x->shape[x->rank - 1], M = t_numel(x) / pitch;
    RCU_REQUIRE(dev, x_col + K <= pitch, "linear: columns [%u, %llu) of rows of %llu", x_col, (unsigned long long)(x_col + K), (unsigned long long)pitch);
    RCU_REQUIRE(dev, t_numel(dst) == M * N, "linear: dst holds %llu elements, expected %llu", (unsigned long long)t_numel(dst), (unsigned long long)(M * N));
    RCU_REQUIRE(dev, !bias || (t_numel(bias) == N && bias->dt == dst->dt), "linear: bias must be a vector of N in the output dtype");
    RCU_REQUIRE(dev, dst->dt == RCU_F32 || (!resid && alpha == 1.0f), "linear: a residual or a factor needs an f32 output");
    RCU_REQUIRE(dev, !resid || (resid->dt == RCU_F32 && t_numel(resid) == M * N), "linear: the residual must be f32 of the output's size");
    RCU_REQUIRE(dev, M <= 0x7fffffffull && N <= 0x7fffffffull && K <= 0x7fffffffull, "linear: dimension exceeds 2^31");
    RCU_REQUIRE(dev, act >= RCU_ACT_NONE && act <= RCU_ACT_SOFTCAP && (act != RCU_ACT_SOFTCAP || act_param > 0.f), "linear: unknown activation %d", act);
    RCU_REQUIRE(dev, act_cols <= N, "linear: %u activated of %llu columns", act_cols, (unsigned long long)N);
    LinearAct fn;
    if (act != RCU_ACT_NONE) { fn.cols = (int)act_cols; fn.kind = act; fn.param = act_param; }
    DevGuard g(dev->ordinal);
    const void* xp = (const char*)x->data + (size_t)x_col * dt_esize(x->dt);
    const void* bp = bias ? bias->data : nullptr;
    const float* rp = resid ? (const float*)resid->data : nullptr;
    if (x->dt != RCU_F32 && M > (uint64_t)kSkinny) {
        TcLinear t;
        t.bf16 = x->dt == RCU_BF16;
        t.x_pitch = pitch;
        t.out_dt = dst->dt;
        t.resid = rp;
        t.alpha = alpha;
        t.act = fn;
        const rcu_status st = rcu_gemm_tc_linear(dev, w->data, xp, bp, dst->data, M, N, K, t);
        if (st != RCU_ERR_UNSUPPORTED) return st;
    }
#define RCU_LIN(T_, O_) return launch_plain<T_, O_>(dev, w->data, xp, pitch, bp, rp, alpha, fn, dst->data, M, N, K)
    if (x->dt == RCU_F32) RCU_LIN(float, float);
    if (x->dt == RCU_BF16) { if (dst->dt == RCU_F32) RCU_LIN(__nv_bfloat16, float); RCU_LIN(__nv_bfloat16, __nv_bfloat16); }
    if (dst->dt == RCU_F32) RCU_LIN(__half, float);
    RCU_LIN(__half, __half);
#undef RCU_LIN
}
