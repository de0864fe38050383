// Latent attention over a block of tokens with a sliding window: what a layer caches per token is one normalised latent
// and one rotated key part shared by all heads, and a head's keys and values are linear images of the latent.
//
//   rcu_latent_append   normalises and rotates the block's latents, keeps the last `ring` of them in the layer's ring
//                       (row of position p: p mod ring) and lays out the rows the block can see;
//   rcu_window_attention  softmax attention of the block's queries over those rows, keys and values expanded from the
//                       latents by one Linear before the call.  bf16 blocks run on the tensor cores (256 tokens and more: window_tc.cu,
//                       fewer, or sizes it does not take: below), f32 ones in FFMA.
// The attention kernels also serve grouped heads with chunked masks and sinks (grouped_attention.cu).
#include "lm_mma.cuh"
#include "window.cuh"

namespace {

struct AppendArgs {
    const float* x;            // [T, pitch], latent at column 0 of the pointer, key part behind it
    long long pitch;
    const float* scale;
    const float* freqs;
    float magnitude, eps;
    int C, R, pairs, T, L, ring;
    uint32_t pos;              // position of the block's first token
};

// rows [0, L - T) of the window come from the ring, the others from the block; one warp per row
template <class O>
__global__ void __launch_bounds__(128) latent_window_kernel(const AppendArgs a, const O* __restrict__ ring, O* __restrict__ out) {
    rcu_kernel_entry();
    const int lane = threadIdx.x & 31;
    const int r = blockIdx.x * 4 + (threadIdx.x >> 5);
    if (r >= a.L) return;
    const int W = a.C + a.R, old = a.L - a.T;
    O* orow = out + (size_t)r * W;
    if (r < old) {
        const O* src = ring + (size_t)((a.pos - (uint32_t)(old - r)) % (uint32_t)a.ring) * W;
        for (int j = lane; j < W; j += 32) orow[j] = src[j];
        return;
    }
    const float* x = a.x + (long long)(r - old) * a.pitch;
    constexpr int kKept = 16;              // elements per lane kept in registers between the two passes
    float v[kKept];
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < kKept; ++i) {
        v[i] = lane + 32 * i < a.C ? x[lane + 32 * i] : 0.f;
        s = fmaf(v[i], v[i], s);
    }
    for (int j = lane + 32 * kKept; j < a.C; j += 32) s = fmaf(x[j], x[j], s);
    const float rstd = 1.0f / sqrtf(warp_sum(s) / (float)a.C + a.eps);
#pragma unroll
    for (int i = 0; i < kKept; ++i)
        if (lane + 32 * i < a.C) orow[lane + 32 * i] = from_f32<O>(v[i] * rstd * a.scale[lane + 32 * i]);
    for (int j = lane + 32 * kKept; j < a.C; j += 32) orow[j] = from_f32<O>(x[j] * rstd * a.scale[j]);
    const float* kr = x + a.C;
    const uint32_t p = a.pos + (uint32_t)(r - old);
    for (int i = lane; i < a.pairs; i += 32) {
        const float2 cs = lm::rotary_angle(a.freqs, a.pairs, i, p, a.magnitude);
        const float u = kr[2 * i], v = kr[2 * i + 1];
        orow[a.C + 2 * i] = from_f32<O>(u * cs.x - v * cs.y);
        orow[a.C + 2 * i + 1] = from_f32<O>(v * cs.x + u * cs.y);
    }
    for (int j = 2 * a.pairs + lane; j < a.R; j += 32) orow[a.C + j] = from_f32<O>(kr[j]);
}

// the block's last min(T, ring) rows into the ring
template <class O>
__global__ void __launch_bounds__(128) latent_store_kernel(const O* __restrict__ rows, O* __restrict__ ring, int W, int n, int L, int ring_rows, uint32_t end) {
    rcu_kernel_entry();
    const int lane = threadIdx.x & 31;
    const int i = blockIdx.x * 4 + (threadIdx.x >> 5);
    if (i >= n) return;
    const O* src = rows + (size_t)(L - n + i) * W;
    O* dst = ring + (size_t)((end - (uint32_t)(n - i)) % (uint32_t)ring_rows) * W;
#pragma unroll 8
    for (int j = lane; j < W; j += 32) dst[j] = src[j];
}

template <class O>
rcu_status launch_append(rcu_device* dev, const AppendArgs& a, void* ring, void* out) {
    rcu_launch(dev, latent_window_kernel<O>, (unsigned)((a.L + 3) / 4), 128, 0, a, (const O*)ring, (O*)out);
    dev->launches++;
    const int n = a.T < a.ring ? a.T : a.ring;
    rcu_launch(dev, latent_store_kernel<O>, (unsigned)((n + 3) / 4), 128, 0, (const O*)out, (O*)ring, a.C + a.R, n, a.L, a.ring, a.pos + (uint32_t)a.T);
    RCU_LAUNCH_CHECK(dev);
    return RCU_OK;
}

// A warp per (token, head): scores 32 keys at a time, one key per lane, online softmax in f32; the weighted sum of the
// values runs over lanes = value columns.
template <class T, int PE>
__global__ void __launch_bounds__(256) window_attention_kernel(const WindowArgs a) {
    rcu_kernel_entry();
    extern __shared__ float q_s[];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int h = blockIdx.y, hk = h / (a.H / a.G);
    const int i = blockIdx.x * 8 + warp;
    if (i >= a.T) return;
    const int Q = a.D + a.R;
    float* q = q_s + warp * Q;
    const T* qg = reinterpret_cast<const T*>(a.q) + ((size_t)i * a.H + h) * Q;
    for (int d = lane; d < Q; d += 32) q[d] = to_f32<T>(qg[d]);
    __syncwarp();
    const size_t kv_pitch = (size_t)a.G * (a.D + a.E);
    const T* K = reinterpret_cast<const T*>(a.kv) + (size_t)hk * a.D;
    const T* V = reinterpret_cast<const T*>(a.kv) + (size_t)a.G * a.D + (size_t)hk * a.E;
    const T* KS = reinterpret_cast<const T*>(a.shared);
    const int last = a.L - a.T + i, first = a.see.first(last);
    float m = -INFINITY, l = 0.f, o[PE];
#pragma unroll
    for (int j = 0; j < PE; ++j) o[j] = 0.f;
    for (int j0 = first; j0 <= last; j0 += 32) {
        const int j = j0 + lane;
        float s = -INFINITY;
        if (j <= last) {
            const T* k = K + j * kv_pitch;
            const T* ks = KS + j * a.shared_pitch;
            float acc = 0.f;
            for (int d = 0; d < a.D; ++d) acc = fmaf(q[d], to_f32<T>(k[d]), acc);
            for (int d = 0; d < a.R; ++d) acc = fmaf(q[a.D + d], to_f32<T>(ks[d]), acc);
            s = acc * a.scale;
        }
        const float mn = fmaxf(m, warp_max(s));
        const float corr = expf(m - mn);
        const float p = expf(s - mn);          // 0 for lanes beyond the last key
        l = l * corr + warp_sum(p);
        m = mn;
#pragma unroll
        for (int c = 0; c < PE; ++c) o[c] *= corr;
        const int n = min(32, last - j0 + 1);
        for (int t = 0; t < n; ++t) {
            const float pt = __shfl_sync(0xffffffffu, p, t);
            const T* v = V + (size_t)(j0 + t) * kv_pitch;
#pragma unroll
            for (int c = 0; c < PE; ++c) {
                const int e = lane + 32 * c;
                if (e < a.E) o[c] = fmaf(pt, to_f32<T>(v[e]), o[c]);
            }
        }
    }
    if (a.sink) l += expf(a.sink[h] - m);
    T* og = reinterpret_cast<T*>(a.out) + ((size_t)i * a.H + h) * a.E;
#pragma unroll
    for (int c = 0; c < PE; ++c) {
        const int e = lane + 32 * c;
        if (e < a.E) og[e] = from_f32<T>(o[c] / l);
    }
}

template <class T> rcu_status launch_window(rcu_device* dev, const WindowArgs& a) {
    const dim3 grid((a.T + 7) / 8, a.H);
    const size_t smem = (size_t)8 * (a.D + a.R) * 4;
#define RCU_WA(PE_)                                                                                                                              \
    do {                                                                                                                                         \
        if (smem > 40 * 1024) RCU_CUDA(dev, cudaFuncSetAttribute(window_attention_kernel<T, PE_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
        rcu_launch(dev, window_attention_kernel<T, PE_>, grid, 256, smem, a);                                                                    \
    } while (0)
    if (a.E <= 64) RCU_WA(2);
    else if (a.E <= 128) RCU_WA(4);
    else if (a.E <= 256) RCU_WA(8);
    else RCU_WA(16);
#undef RCU_WA
    RCU_LAUNCH_CHECK(dev);
    return RCU_OK;
}

// Tensor-core form for bf16: CTA = (128 queries, head), a warp per 16 queries; keys and values 64 at a time through two
// asynchronous stages in shared memory.  Scores, softmax and the output sums are f32; the weights enter the product with the
// values as bf16 value plus remainder.
constexpr int kQueries = 128, kKeys = 64;

template <int EP>
__global__ void __launch_bounds__(256) window_mma_kernel(const WindowArgs a, int vec) {
    rcu_kernel_entry();
    using lm::bf16;
    extern __shared__ __align__(16) bf16 tiles[];
    const int Q = a.D + a.R, qp = (Q + 15) & ~15, ld = qp + 8;
    constexpr int ldv = EP + 8;
    bf16 *qs = tiles, *ks = qs + kQueries * ld, *vs = ks + 2 * kKeys * ld;
    const int h = blockIdx.y, hk = h / (a.H / a.G), i0 = blockIdx.x * kQueries;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int nq = min(kQueries, a.T - i0);
    const long long kvp = (long long)a.G * (a.D + a.E);
    const bf16* K = reinterpret_cast<const bf16*>(a.kv) + (size_t)hk * a.D;
    const bf16* V = reinterpret_cast<const bf16*>(a.kv) + (size_t)a.G * a.D + (size_t)hk * a.E;
    const bf16* KS = reinterpret_cast<const bf16*>(a.shared);
    const int base = a.L - a.T + i0;                       // key row of the CTA's first query
    const int first = a.see.first(base), last = base + nq - 1;
    const int tiles_n = (last - first) / kKeys + 1;

    auto load_keys = [&](int n) {
        const int j0 = first + n * kKeys, rows = min(kKeys, last + 1 - j0);
        bf16* kt = ks + (n & 1) * kKeys * ld;
        if (vec) {
            lm::load_tile(kt, ld, K + (long long)j0 * kvp, kvp, kKeys, rows, a.D, a.D, true);
            lm::load_tile(kt + a.D, ld, KS + (long long)j0 * a.shared_pitch, a.shared_pitch, kKeys, rows, a.R, a.R, true);
        } else {
            for (int i = threadIdx.x; i < kKeys * Q; i += 256) {
                const int r = i / Q, c = i - r * Q;
                const bf16* s = c < a.D ? K + (long long)(j0 + r) * kvp + c : KS + (long long)(j0 + r) * a.shared_pitch + c - a.D;
                kt[r * ld + c] = r < rows ? *s : __float2bfloat16_rn(0.f);
            }
        }
        lm::load_tile(vs + (n & 1) * kKeys * ldv, ldv, V + (long long)j0 * kvp, kvp, kKeys, rows, a.E, EP, vec);
        lm::cp_commit();
    };
    // columns between the head's features and the next multiple of 16 stay zero
    for (int i = threadIdx.x; i < (kQueries + 2 * kKeys) * (qp - Q); i += 256) {
        const int r = i / (qp - Q);
        (r < kQueries ? qs + r * ld : ks + (r - kQueries) * ld)[Q + i % (qp - Q)] = __float2bfloat16_rn(0.f);
    }
    const bf16* qg = reinterpret_cast<const bf16*>(a.q) + ((size_t)i0 * a.H + h) * Q;
    if (vec) {
        lm::load_tile(qs, ld, qg, (long long)a.H * Q, kQueries, nq, Q, Q, true);
    } else {
        for (int i = threadIdx.x; i < kQueries * Q; i += 256) {
            const int r = i / Q, c = i - r * Q;
            qs[r * ld + c] = r < nq ? qg[(size_t)r * a.H * Q + c] : __float2bfloat16_rn(0.f);
        }
    }
    load_keys(0);

    const int r0 = warp * 16, row0 = base + r0 + g, row1 = row0 + 8;      // key rows of this thread's two queries
    const int low0 = a.see.first(row0), low1 = a.see.first(row1), low = a.see.first(base + r0);
    const float sc = a.scale * 1.4426950408889634f;                       // scores in units of log 2
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f, o[EP / 8][4];
#pragma unroll
    for (int j = 0; j < EP / 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;

    for (int n = 0; n < tiles_n; ++n) {
        if (n + 1 < tiles_n) {
            load_keys(n + 1);
            lm::cp_wait<1>();
        } else {
            lm::cp_wait<0>();
        }
        __syncthreads();
        const int j0 = first + n * kKeys;
        // a tile no query of this warp sees is passed over
        if (r0 < nq && j0 <= base + r0 + 15 && j0 + kKeys - 1 >= low) {
            const bf16* kt = ks + (n & 1) * kKeys * ld;
            const bf16* vt = vs + (n & 1) * kKeys * ldv;
            float s[8][4] = {};
            for (int k0 = 0; k0 < qp; k0 += 16) {
                uint32_t qa[4];
                lm::load_a(qa, qs, ld, r0, k0);
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    uint32_t b[4];
                    lm::load_b(b, kt, ld, 16 * c, k0);
                    lm::mma(s[2 * c], qa, b[0], b[1]);
                    lm::mma(s[2 * c + 1], qa, b[2], b[3]);
                }
            }
            float t0 = -INFINITY, t1 = -INFINITY;
#pragma unroll
            for (int c = 0; c < 8; ++c)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int j = j0 + 8 * c + 2 * t + (e & 1);
                    const float v = j <= (e < 2 ? row0 : row1) && j >= (e < 2 ? low0 : low1) ? s[c][e] * sc : -INFINITY;
                    s[c][e] = v;
                    if (e < 2) t0 = fmaxf(t0, v);
                    else t1 = fmaxf(t1, v);
                }
            t0 = fmaxf(t0, __shfl_xor_sync(0xffffffffu, t0, 1));
            t1 = fmaxf(t1, __shfl_xor_sync(0xffffffffu, t1, 1));
            t0 = fmaxf(t0, __shfl_xor_sync(0xffffffffu, t0, 2));
            t1 = fmaxf(t1, __shfl_xor_sync(0xffffffffu, t1, 2));
            const float n0 = fmaxf(m0, t0), n1 = fmaxf(m1, t1);
            const float z0 = n0 == -INFINITY ? 0.f : n0, z1 = n1 == -INFINITY ? 0.f : n1;      // no key seen yet: weights of zero
            const float c0 = exp2f(m0 - z0), c1 = exp2f(m1 - z1);
            m0 = n0; m1 = n1;
            l0 *= c0; l1 *= c1;
#pragma unroll
            for (int c = 0; c < 8; ++c) {
                s[c][0] = exp2f(s[c][0] - z0); s[c][1] = exp2f(s[c][1] - z0);
                s[c][2] = exp2f(s[c][2] - z1); s[c][3] = exp2f(s[c][3] - z1);
                l0 += s[c][0] + s[c][1];
                l1 += s[c][2] + s[c][3];
            }
#pragma unroll
            for (int j = 0; j < EP / 8; ++j) { o[j][0] *= c0; o[j][1] *= c0; o[j][2] *= c1; o[j][3] *= c1; }
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) {
                uint32_t ph[4], pl[4];
                lm::split2(s[2 * kk][0], s[2 * kk][1], ph[0], pl[0]);
                lm::split2(s[2 * kk][2], s[2 * kk][3], ph[1], pl[1]);
                lm::split2(s[2 * kk + 1][0], s[2 * kk + 1][1], ph[2], pl[2]);
                lm::split2(s[2 * kk + 1][2], s[2 * kk + 1][3], ph[3], pl[3]);
#pragma unroll
                for (int j = 0; j < EP / 16; ++j) {
                    uint32_t b[4];
                    lm::load_b_t(b, vt, ldv, 16 * j, 16 * kk);
                    lm::mma(o[2 * j], ph, b[0], b[1]);
                    lm::mma(o[2 * j + 1], ph, b[2], b[3]);
                    lm::mma(o[2 * j], pl, b[0], b[1]);
                    lm::mma(o[2 * j + 1], pl, b[2], b[3]);
                }
            }
        }
        __syncthreads();
    }
    l0 += __shfl_xor_sync(0xffffffffu, l0, 1);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
    l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
    if (a.sink) {
        const float sink = a.sink[h] * 1.4426950408889634f;
        l0 += exp2f(sink - m0);
        l1 += exp2f(sink - m1);
    }
    const float w0 = 1.0f / l0, w1 = 1.0f / l1;
    bf16* og = reinterpret_cast<bf16*>(a.out) + (size_t)i0 * a.H * a.E + (size_t)h * a.E;
#pragma unroll
    for (int j = 0; j < EP / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int r = r0 + g + (e < 2 ? 0 : 8), c = 8 * j + 2 * t + (e & 1);
            if (r < nq && c < a.E) og[(size_t)r * a.H * a.E + c] = __float2bfloat16_rn(o[j][e] * (e < 2 ? w0 : w1));
        }
}

size_t window_mma_smem(int Q, int EP) { return ((size_t)(kQueries + 2 * kKeys) * (((Q + 15) & ~15) + 8) + 2 * (size_t)kKeys * (EP + 8)) * sizeof(lm::bf16); }

rcu_status launch_window_mma(rcu_device* dev, const WindowArgs& a) {
    const int Q = a.D + a.R, ep = a.E <= 32 ? 32 : a.E <= 64 ? 64 : a.E <= 128 ? 128 : 256;
    if (a.E > 256 || window_mma_smem(Q, ep) > (size_t)dev->smem_optin) return RCU_ERR_UNSUPPORTED;
    const size_t smem = window_mma_smem(Q, ep);
    const int vec = a.D % 8 == 0 && a.R % 8 == 0 && a.E % 8 == 0 && a.shared_pitch % 8 == 0 &&
                    ((reinterpret_cast<uintptr_t>(a.q) | reinterpret_cast<uintptr_t>(a.kv) | reinterpret_cast<uintptr_t>(a.shared)) & 15) == 0;
    const dim3 grid((a.T + kQueries - 1) / kQueries, a.H);
#define RCU_WM(EP_)                                                                                                          \
    do {                                                                                                                     \
        RCU_CUDA(dev, cudaFuncSetAttribute(window_mma_kernel<EP_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
        rcu_launch(dev, window_mma_kernel<EP_>, grid, 256, smem, a, vec);                                                    \
    } while (0)
    if (ep == 32) RCU_WM(32);
    else if (ep == 64) RCU_WM(64);
    else if (ep == 128) RCU_WM(128);
    else RCU_WM(256);
#undef RCU_WM
    RCU_LAUNCH_CHECK(dev);
    return RCU_OK;
}

}  // namespace

rcu_status rcu_attend(rcu_device* dev, int dt, const WindowArgs& a) {
    if (dt == RCU_F32) return launch_window<float>(dev, a);
    rcu_status st = rcu_window_tc(dev, a);
    if (st == RCU_ERR_UNSUPPORTED) st = launch_window_mma(dev, a);
    return st == RCU_ERR_UNSUPPORTED ? launch_window<__nv_bfloat16>(dev, a) : st;
}

extern "C" {

rcu_status rcu_latent_append(rcu_device* dev, const rcu_tensor* x, uint32_t x_col, const rcu_tensor* scale, float eps, const rcu_tensor* freqs,
                             float magnitude, uint32_t position, rcu_tensor* ring, rcu_tensor* dst) {
    if (!dev) return RCU_ERR_INVALID_ARG;
    RCU_REQUIRE(dev, t_valid(x) && t_valid(scale) && t_valid(freqs) && t_valid(ring) && t_valid(dst), "latent_append: invalid tensor descriptor");
    RCU_REQUIRE(dev, x->dt == RCU_F32 && scale->dt == RCU_F32 && freqs->dt == RCU_F32, "latent_append: f32 rows, scale and frequencies");
    RCU_REQUIRE(dev, ring->rank == 2 && dst->rank == 2 && ring->dt == dst->dt && (ring->dt == RCU_F32 || ring->dt == RCU_BF16) &&
                         ring->shape[1] == dst->shape[1], "latent_append: ring and dst are f32 or bf16 rows of one width");
    RCU_REQUIRE(dev, freqs->rank == 2 && freqs->shape[0] == 2, "latent_append: the frequency table is f32 [2, pairs]");
    const uint64_t W = ring->shape[1], C = t_numel(scale), pitch = x->shape[x->rank - 1], T = t_numel(x) / pitch, L = dst->shape[0];
    RCU_REQUIRE(dev, C < W && x_col + W <= pitch && 2 * freqs->shape[1] <= W - C, "latent_append: columns do not fit the rows");
    RCU_REQUIRE(dev, L >= T && L - T <= position && L - T <= ring->shape[0] && L <= 0x7fffffffull, "latent_append: the window reaches before the ring");
    DevGuard g(dev->ordinal);
    AppendArgs a{(const float*)x->data + x_col, (long long)pitch, (const float*)scale->data, (const float*)freqs->data, magnitude, eps, (int)C, (int)(W - C),
                 (int)freqs->shape[1], (int)T, (int)L, (int)ring->shape[0], position};
    return ring->dt == RCU_F32 ? launch_append<float>(dev, a, ring->data, dst->data) : launch_append<__nv_bfloat16>(dev, a, ring->data, dst->data);
}

rcu_status rcu_window_attention(rcu_device* dev, const rcu_tensor* q, const rcu_tensor* kv, const rcu_tensor* shared, uint32_t shared_col, uint32_t vdim,
                                uint32_t window, float scale, rcu_tensor* dst) {
    if (!dev) return RCU_ERR_INVALID_ARG;
    RCU_REQUIRE(dev, t_valid(q) && t_valid(kv) && t_valid(shared) && t_valid(dst), "window_attention: invalid tensor descriptor");
    RCU_REQUIRE(dev, q->rank == 3 && kv->rank == 2 && shared->rank == 2 && q->dt == kv->dt && q->dt == shared->dt && q->dt == dst->dt &&
                         (q->dt == RCU_F32 || q->dt == RCU_BF16), "window_attention: q [tokens, heads, dim], kv and shared rows, f32 or bf16");
    const uint64_t T = q->shape[0], H = q->shape[1], L = kv->shape[0];
    RCU_REQUIRE(dev, vdim > 0 && window > 0 && shared_col <= shared->shape[1] && shared->shape[0] == L && L >= T, "window_attention: bad sizes");
    const uint64_t R = shared->shape[1] - shared_col;
    RCU_REQUIRE(dev, q->shape[2] >= R && kv->shape[1] == H * (q->shape[2] - R + vdim), "window_attention: kv rows hold every head's keys, then its values");
    RCU_REQUIRE(dev, t_numel(dst) == T * H * vdim, "window_attention: dst holds %llu elements, expected %llu", (unsigned long long)t_numel(dst),
                (unsigned long long)(T * H * vdim));
    if (vdim > 512 || H > 65535 || L > 0x7fffffffull || q->shape[2] > 4096) return rcu_fail(dev, RCU_ERR_UNSUPPORTED, "window_attention: vdim %u (at most 512)", vdim);
    DevGuard g(dev->ordinal);
    WindowArgs a{q->data, kv->data, (const char*)shared->data + (size_t)shared_col * dt_esize(shared->dt), dst->data, (long long)shared->shape[1], (int)T,
                 (int)L, (int)H, (int)H, (int)(q->shape[2] - R), (int)R, (int)vdim, Visible{(int)(window < L ? window : L), 0, 0}, scale, nullptr};
    return rcu_attend(dev, q->dt, a);
}

}  // extern "C"
