// Attention of grouped heads over a block of tokens: keys and values of kv_heads heads are cached per layer in a ring of rows
// (position p in row p mod ring rows), queries and keys are normed per head and rotated, and a query sees a run of the rows that ends
// with itself - a sliding window, or the chunk of positions it lies in.
//
//   rcu_kv_append          norms and rotates the block's keys, lays out the rows the block can see (older ones from the ring) and keeps
//                          its last rows in the ring;
//   rcu_grouped_attention  softmax attention with an optional sink over those rows, on the kernels of latent_attention.cu and
//                          window_tc.cu.
#include "head_norm.cuh"
#include "window.cuh"

namespace {

struct KvArgs {
    lm::HeadNorm norm;
    long long pitch;           // of the block's rows
    int G, E, T, L, ring_rows, keep, direct;      // direct: this kernel also writes the ring
    uint32_t pos;              // position of the block's first token
};

constexpr int kKvHeads = 2;           // kv heads of a row that a group of lanes takes

// A group of lanes per (row, kKvHeads kv heads), or (V == 1) a warp per (row, kv head): rows [0, L - T) come from the ring, the
// others from the block.
template <class T, int V>
__global__ void __launch_bounds__(256) kv_rows_kernel(const KvArgs a, const T* __restrict__ x, T* ring, T* __restrict__ out, long long n, int lanes) {
    rcu_kernel_entry();
    using Vec = lm::HeadVec<T, V>;
    constexpr int N = V == 1 ? 1 : kKvHeads;
    const int lane = threadIdx.x & 31, s = lane & (lanes - 1), D = a.norm.dim, per = (a.G + N - 1) / N;
    const long long item = ((long long)blockIdx.x * 8 + (threadIdx.x >> 5)) * (32 / lanes) + lane / lanes;
    const bool live = item < n;
    const int r = live ? (int)(item / per) : 0, g = live ? (int)(item - (long long)r * per) * N : 0, heads = live ? min(N, a.G - g) : 0;
    const int old = a.L - a.T, t = r - old;
    const long long W = (long long)a.G * (D + a.E), kc = (long long)g * D, vc = (long long)a.G * D + (long long)g * a.E;
    T* orow = out + r * W;
    const bool fresh = live && t >= 0;
    const T* src = fresh ? x + t * a.pitch : ring + (size_t)((a.pos - (uint32_t)(old - r)) % (uint32_t)a.ring_rows) * W;
    T* store = fresh && a.direct && t >= a.T - a.keep ? ring + (size_t)((a.pos + (uint32_t)t) % (uint32_t)a.ring_rows) * W : nullptr;
    if constexpr (V == 1) {
        lm::head_norm_rotate<T>(a.norm, fresh ? src + kc : x, fresh ? t : 0, orow + kc, store ? store + kc : nullptr, s, fresh);
        if (live && !fresh)
            for (int c = s; c < D; c += 32) orow[kc + c] = src[kc + c];
    } else {
        lm::HeadPart<T, V> part;
        part.load(a.norm, fresh ? t : 0, s, live);
        Vec k[N];
#pragma unroll
        for (int j = 0; j < N; ++j) k[j] = part.in && j < heads ? *reinterpret_cast<const Vec*>(src + kc + j * D + part.c) : Vec{};
#pragma unroll
        for (int j = 0; j < N; ++j) {
            const Vec y = part.apply(a.norm, k[j], lanes);
            if (fresh) k[j] = y;
            if (part.in && j < heads) {
                *reinterpret_cast<Vec*>(orow + kc + j * D + part.c) = k[j];
                if (store) *reinterpret_cast<Vec*>(store + kc + j * D + part.c) = k[j];
            }
        }
    }
    // the values of these heads lie side by side
#pragma unroll 4
    for (int c = s * V; c < heads * a.E; c += lanes * V) {
        const Vec v = *reinterpret_cast<const Vec*>(src + vc + c);
        *reinterpret_cast<Vec*>(orow + vc + c) = v;
        if (store) *reinterpret_cast<Vec*>(store + vc + c) = v;
    }
}

// the block's last n rows into the ring, for blocks whose rows would overwrite older ones that are still to be read
template <class Unit>
__global__ void __launch_bounds__(256) kv_store_kernel(const Unit* __restrict__ rows, Unit* __restrict__ ring, int units, int n, int L, int ring_rows, uint32_t end) {
    rcu_kernel_entry();
    const int lane = threadIdx.x & 31, i = blockIdx.x * 8 + (threadIdx.x >> 5);
    if (i >= n) return;
    const Unit* src = rows + (size_t)(L - n + i) * units;
    Unit* dst = ring + (size_t)((end - (uint32_t)(n - i)) % (uint32_t)ring_rows) * units;
#pragma unroll 4
    for (int j = lane; j < units; j += 32) dst[j] = src[j];
}

template <class T>
rcu_status launch_kv_append(rcu_device* dev, KvArgs a, const void* x, void* ring, void* out) {
    constexpr int V = 16 / (int)sizeof(T);
    const int D = a.norm.dim, old = a.L - a.T;
    const size_t W = (size_t)a.G * (D + a.E);
    // the rows read and the rows written are different ones when together they fit the ring
    a.direct = a.keep > 0 && (old == 0 || a.L <= a.ring_rows);
    const bool aligned = ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(ring) | reinterpret_cast<uintptr_t>(out) |
                           reinterpret_cast<uintptr_t>(a.norm.scale) | reinterpret_cast<uintptr_t>(a.norm.angles)) & 15) == 0;
    const bool vec = D % V == 0 && a.E % V == 0 && D <= 32 * V && a.pitch % V == 0 && aligned;
    const int lanes = vec ? lm::head_lanes(D, V) : 32, per = 8 * (32 / lanes);
    const long long n = (long long)a.L * (vec ? (a.G + kKvHeads - 1) / kKvHeads : a.G);
    const unsigned grid = (unsigned)((n + per - 1) / per);
    if (vec) rcu_launch(dev, kv_rows_kernel<T, V>, grid, 256, 0, a, (const T*)x, (T*)ring, (T*)out, n, lanes);
    else rcu_launch(dev, kv_rows_kernel<T, 1>, grid, 256, 0, a, (const T*)x, (T*)ring, (T*)out, n, lanes);
    RCU_LAUNCH_CHECK(dev);
    if (a.keep > 0 && !a.direct) {
        const unsigned blocks = (unsigned)((a.keep + 7) / 8);
        const uint32_t end = a.pos + (uint32_t)a.T;
        if (W % V == 0 && aligned)
            rcu_launch(dev, kv_store_kernel<uint4>, blocks, 256, 0, (const uint4*)out, (uint4*)ring, (int)(W / V), a.keep, a.L, a.ring_rows, end);
        else
            rcu_launch(dev, kv_store_kernel<T>, blocks, 256, 0, (const T*)out, (T*)ring, (int)W, a.keep, a.L, a.ring_rows, end);
        RCU_LAUNCH_CHECK(dev);
    }
    return RCU_OK;
}

}  // namespace

extern "C" {

rcu_status rcu_kv_append(rcu_device* dev, const rcu_tensor* x, uint32_t x_col, uint32_t kv_heads, const rcu_tensor* scale, float eps, const rcu_tensor* angles,
                         uint32_t position, uint32_t keep, rcu_tensor* ring, rcu_tensor* dst) {
    if (!dev) return RCU_ERR_INVALID_ARG;
    RCU_REQUIRE(dev, t_valid(x) && t_valid(scale) && t_valid(angles) && t_valid(ring) && t_valid(dst), "kv_append: invalid tensor descriptor");
    RCU_REQUIRE(dev, x->rank == 2 && ring->rank == 2 && dst->rank == 2 && angles->rank == 2 && x->dt == ring->dt && x->dt == dst->dt &&
                         (x->dt == RCU_F32 || x->dt == RCU_BF16) && scale->dt == RCU_F32 && angles->dt == RCU_F32, "kv_append: f32 or bf16 rows of one dtype");
    const uint64_t T = x->shape[0], L = dst->shape[0], W = ring->shape[1], D = t_numel(scale);
    RCU_REQUIRE(dev, kv_heads > 0 && W % kv_heads == 0 && W / kv_heads > D && dst->shape[1] == W && x_col + W <= x->shape[1], "kv_append: bad row widths");
    RCU_REQUIRE(dev, angles->shape[0] == T && angles->shape[1] <= D && D <= 65536, "kv_append: angles are [tokens, 2 pairs] of at most dim features");
    RCU_REQUIRE(dev, L >= T && L - T <= position && L - T <= ring->shape[0] && L * kv_heads <= 0x7fffffffull, "kv_append: the visible rows reach before the ring");
    RCU_REQUIRE(dev, keep <= T && keep <= ring->shape[0] && ring->shape[0] <= 0x7fffffffull, "kv_append: %u rows to keep of %llu in %llu", keep, (unsigned long long)T,
                (unsigned long long)ring->shape[0]);
    DevGuard g(dev->ordinal);
    KvArgs a{{(const float*)scale->data, (const float*)angles->data, (int)D, (int)(angles->shape[1] / 2), eps}, (long long)x->shape[1], (int)kv_heads,
             (int)(W / kv_heads - D), (int)T, (int)L, (int)ring->shape[0], (int)keep, 0, position};
    const void* xp = (const char*)x->data + (size_t)x_col * dt_esize(x->dt);
    return x->dt == RCU_F32 ? launch_kv_append<float>(dev, a, xp, ring->data, dst->data) : launch_kv_append<__nv_bfloat16>(dev, a, xp, ring->data, dst->data);
}

rcu_status rcu_grouped_attention(rcu_device* dev, const rcu_tensor* q, const rcu_tensor* kv, const rcu_tensor* sink, uint32_t kv_heads, uint32_t vdim,
                                 uint32_t window, uint32_t chunk, uint32_t position, float scale, rcu_tensor* dst) {
    if (!dev) return RCU_ERR_INVALID_ARG;
    RCU_REQUIRE(dev, t_valid(q) && t_valid(kv) && (!sink || t_valid(sink)) && t_valid(dst), "grouped_attention: invalid tensor descriptor");
    RCU_REQUIRE(dev, q->rank == 3 && kv->rank == 2 && q->dt == kv->dt && q->dt == dst->dt && (q->dt == RCU_F32 || q->dt == RCU_BF16),
                "grouped_attention: q [tokens, heads, dim] and kv rows, f32 or bf16");
    const uint64_t T = q->shape[0], H = q->shape[1], D = q->shape[2], L = kv->shape[0];
    RCU_REQUIRE(dev, kv_heads > 0 && H % kv_heads == 0 && vdim > 0 && L >= T && kv->shape[1] == kv_heads * (D + vdim), "grouped_attention: kv rows hold every head's keys, then its values");
    RCU_REQUIRE(dev, !sink || (sink->dt == RCU_F32 && t_numel(sink) == H), "grouped_attention: one f32 sink per query head");
    RCU_REQUIRE(dev, t_numel(dst) == T * H * vdim, "grouped_attention: dst holds %llu elements, expected %llu", (unsigned long long)t_numel(dst),
                (unsigned long long)(T * H * vdim));
    RCU_REQUIRE(dev, (uint64_t)position + L < (1u << 30), "grouped_attention: positions up to 2^30");
    if (vdim > 512 || H > 65535 || D > 1024) return rcu_fail(dev, RCU_ERR_UNSUPPORTED, "grouped_attention: heads of %llu and %u (at most 1024 and 512)", (unsigned long long)D, vdim);
    DevGuard g(dev->ordinal);
    const Visible see{window == 0 || window > L ? (int)L : (int)window, chunk > (1u << 30) ? 1 << 30 : (int)chunk, position};
    const WindowArgs a{q->data, kv->data, nullptr, dst->data, 8, (int)T, (int)L, (int)H, (int)kv_heads, (int)D, 0, (int)vdim, see, scale,
                       sink ? (const float*)sink->data : nullptr};
    return rcu_attend(dev, q->dt, a);
}

}  // extern "C"
