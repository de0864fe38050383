// Linear attention with a fixed decay per head ("lightning" attention) over a block of tokens:
//   S_t = d_h S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,
// q, k, v the (optionally silu-activated) columns [0, HD), [HD, 2HD), [2HD, 2HD + HE) of the input rows, S [H, D, E] in
// f32, updated in place.
//
// lightning_recurrent_kernel runs the recurrence token by token in f32 and takes any sizes.
#include "lm_math.cuh"

namespace {

struct LightningArgs {
    const void* x;
    long long pitch;
    const float* decay_pow;    // [H, n_pow]: d_h^0, d_h^1, ...
    int n_pow;
    float* state;
    float* out;                // [T, H * E]
    int T, H, D, E, silu;
};

constexpr int kTok = 8;        // tokens staged at a time

// One CTA per (head, 32 value columns).  Thread (warp g, lane e) keeps S[g + 8 j][e] for all j in registers; the eight
// warps' shares of o_t meet in shared memory once per kTok tokens.
template <class T, int PER>
__global__ void __launch_bounds__(256) lightning_recurrent_kernel(const LightningArgs a) {
    rcu_kernel_entry();
    __shared__ float qs[kTok][PER * 8], ks[kTok][PER * 8], vs[kTok][32];
    __shared__ float part[kTok][8][32];
    const int h = blockIdx.x, e0 = blockIdx.y * 32;
    const int lane = threadIdx.x & 31, g = threadIdx.x >> 5;
    const int e = e0 + lane;
    const float decay = a.decay_pow[(size_t)h * a.n_pow + 1];
    const T* x = reinterpret_cast<const T*>(a.x);
    const long long HD = (long long)a.H * a.D;
    float* S = a.state + (size_t)h * a.D * a.E;
    float s[PER];
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int d = g + 8 * j;
        s[j] = (d < a.D && e < a.E) ? S[(size_t)d * a.E + e] : 0.f;
    }
    auto act = [&](float z) { return a.silu ? lm::silu(z) : z; };
    for (int t0 = 0; t0 < a.T; t0 += kTok) {
        const int n = min(kTok, a.T - t0);
        __syncthreads();
        for (int i = threadIdx.x; i < kTok * PER * 8; i += 256) {
            const int t = i / (PER * 8), d = i % (PER * 8);
            const bool in = t < n && d < a.D;
            const T* row = x + (size_t)(t0 + (in ? t : 0)) * a.pitch + (size_t)h * a.D + (in ? d : 0);
            qs[t][d] = in ? act(to_f32<T>(row[0])) : 0.f;
            ks[t][d] = in ? act(to_f32<T>(row[HD])) : 0.f;
        }
        for (int i = threadIdx.x; i < kTok * 32; i += 256) {
            const int t = i >> 5, c = e0 + (i & 31);
            vs[t][i & 31] = (t < n && c < a.E) ? act(to_f32<T>(x[(size_t)(t0 + t) * a.pitch + 2 * HD + (size_t)h * a.E + c])) : 0.f;
        }
        __syncthreads();
        for (int t = 0; t < n; ++t) {
            const float v = vs[t][lane];
            float o = 0.f;
#pragma unroll
            for (int j = 0; j < PER; ++j) {
                s[j] = fmaf(decay, s[j], ks[t][g + 8 * j] * v);
                o = fmaf(qs[t][g + 8 * j], s[j], o);
            }
            part[t][g][lane] = o;
        }
        __syncthreads();
        for (int i = threadIdx.x; i < n * 32; i += 256) {
            const int t = i >> 5, c = i & 31;
            if (e0 + c >= a.E) continue;
            float o = 0.f;
#pragma unroll
            for (int w = 0; w < 8; ++w) o += part[t][w][c];
            a.out[(size_t)(t0 + t) * a.H * a.E + (size_t)h * a.E + e0 + c] = o;
        }
    }
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int d = g + 8 * j;
        if (d < a.D && e < a.E) S[(size_t)d * a.E + e] = s[j];
    }
}

template <class T> rcu_status launch_recurrent(rcu_device* dev, const LightningArgs& a) {
    const dim3 grid(a.H, (a.E + 31) / 32);
    const int per = (a.D + 7) / 8;
    if (per <= 4) rcu_launch(dev, lightning_recurrent_kernel<T, 4>, grid, 256, 0, a);
    else if (per <= 8) rcu_launch(dev, lightning_recurrent_kernel<T, 8>, grid, 256, 0, a);
    else if (per <= 16) rcu_launch(dev, lightning_recurrent_kernel<T, 16>, grid, 256, 0, a);
    else rcu_launch(dev, lightning_recurrent_kernel<T, 32>, grid, 256, 0, a);
    RCU_LAUNCH_CHECK(dev);
    return RCU_OK;
}

}  // namespace

extern "C" rcu_status rcu_lightning(rcu_device* dev, const rcu_tensor* x, const rcu_tensor* decay_pow, rcu_tensor* state, int silu, rcu_tensor* dst) {
    if (!dev) return RCU_ERR_INVALID_ARG;
    RCU_REQUIRE(dev, t_valid(x) && t_valid(decay_pow) && t_valid(state) && t_valid(dst), "lightning: invalid tensor descriptor");
    RCU_REQUIRE(dev, x->dt == RCU_F32 || x->dt == RCU_BF16, "lightning: f32 or bf16 rows");
    RCU_REQUIRE(dev, state->dt == RCU_F32 && state->rank == 3 && dst->dt == RCU_F32, "lightning: the state is f32 [heads, dim, vdim], the output f32");
    const uint64_t H = state->shape[0], D = state->shape[1], E = state->shape[2];
    const uint64_t pitch = x->shape[x->rank - 1], T = t_numel(x) / pitch;
    RCU_REQUIRE(dev, decay_pow->dt == RCU_F32 && decay_pow->rank == 2 && decay_pow->shape[0] == H && decay_pow->shape[1] >= 2,
                "lightning: decay powers are f32 [heads, >= 2]");
    RCU_REQUIRE(dev, 2 * H * D + H * E <= pitch && t_numel(dst) == T * H * E, "lightning: rows or output do not fit heads x (dim, dim, vdim)");
    if (D > 256 || H > 65535 || E > 65535 * 32ull || T > 0x7fffffffull) return rcu_fail(dev, RCU_ERR_UNSUPPORTED, "lightning: dim %llu (at most 256)", (unsigned long long)D);
    DevGuard g(dev->ordinal);
    LightningArgs a{x->data, (long long)pitch, (const float*)decay_pow->data, (int)decay_pow->shape[1], (float*)state->data, (float*)dst->data,
                    (int)T, (int)H, (int)D, (int)E, silu != 0};
    return x->dt == RCU_F32 ? launch_recurrent<float>(dev, a) : launch_recurrent<__nv_bfloat16>(dev, a);
}
