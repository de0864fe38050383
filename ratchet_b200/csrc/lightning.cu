// Linear attention with a fixed decay per head ("lightning" attention) over a block of tokens:
//   S_t = d_h S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,
// q, k, v the columns [0, HD), [HD, 2HD), [2HD, 2HD + HE) of the input rows, S [H, D, E] in f32, updated in place.
//
// lightning_recurrent_kernel runs the recurrence token by token in f32; it takes any sizes, f32 rows and short blocks.
// Longer blocks of bf16 rows run in chunks of 128 tokens on the tensor cores, in three launches that are each parallel
// over chunks or over state elements:
//   chunk_kv     every chunk's own contribution to the state, U_n = sum_j d^(last - j) k_j v_j^T;
//   chunk_scan   S_(n+1) = d^128 S_n + U_n element by element, leaving S_n where U_n was;
//   chunk_out    o_i = d^(i+1) S_n^T q_i + sum_(j <= i) d^(i-j) (q_i . k_j) v_j.
// The operands that must keep f32 accuracy (decayed keys, states, decayed scores) enter the bf16 products as value plus
// remainder, two products each.
#include <algorithm>

#include "lm_mma.cuh"

namespace {

struct LightningArgs {
    const void* x;
    long long pitch;
    const float* decay_pow;    // [H, n_pow]: d_h^0, d_h^1, ...
    int n_pow;
    float* state;
    float* out;                // [T, H * E]
    int T, H, D, E;
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
    for (int t0 = 0; t0 < a.T; t0 += kTok) {
        const int n = min(kTok, a.T - t0);
        __syncthreads();
        for (int i = threadIdx.x; i < kTok * PER * 8; i += 256) {
            const int t = i / (PER * 8), d = i % (PER * 8);
            const bool in = t < n && d < a.D;
            const T* row = x + (size_t)(t0 + (in ? t : 0)) * a.pitch + (size_t)h * a.D + (in ? d : 0);
            qs[t][d] = in ? to_f32<T>(row[0]) : 0.f;
            ks[t][d] = in ? to_f32<T>(row[HD]) : 0.f;
        }
        for (int i = threadIdx.x; i < kTok * 32; i += 256) {
            const int t = i >> 5, c = e0 + (i & 31);
            vs[t][i & 31] = (t < n && c < a.E) ? to_f32<T>(x[(size_t)(t0 + t) * a.pitch + 2 * HD + (size_t)h * a.E + c]) : 0.f;
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
    else if (per <= 32) rcu_launch(dev, lightning_recurrent_kernel<T, 32>, grid, 256, 0, a);
    else rcu_launch(dev, lightning_recurrent_kernel<T, 64>, grid, 256, 0, a);
    RCU_LAUNCH_CHECK(dev);
    return RCU_OK;
}

// ---------------------------------------------------------------------------------------- chunks on the tensor cores
constexpr int kChunk = 128;
constexpr int kTile = 64;                      // state rows / columns per CTA tile
constexpr int kLdT = kTile + 8;                // row pitch of a 64-wide bf16 tile: rows start in different banks

struct ChunkArgs {
    const lm::bf16* x;
    long long pitch;
    const float* decay_pow;
    int n_pow;
    float* state;
    uint32_t* scratch;                         // [chunks, H, D, E]: U as f32, then S as bf16 value (high half) and remainder
    float* out;
    int T, H, D, E, vec;
};

// two neighbouring elements of a row of n (e is even, and so is the row's offset where n is)
__device__ __forceinline__ void store2(float* row, int e, int n, float x, float y) {
    if (n % 2 == 0 && e < n) *reinterpret_cast<float2*>(row + e) = make_float2(x, y);
    else {
        if (e < n) row[e] = x;
        if (e + 1 < n) row[e + 1] = y;
    }
}

__global__ void __launch_bounds__(128) chunk_kv_kernel(const ChunkArgs a) {
    rcu_kernel_entry();
    extern __shared__ __align__(16) lm::bf16 tiles[];
    lm::bf16 *kh = tiles, *kl = kh + kChunk * kLdT, *vs = kl + kChunk * kLdT;
    const int n = blockIdx.x, h = blockIdx.y, te = (a.E + kTile - 1) / kTile;
    const int d0 = (blockIdx.z / te) * kTile, e0 = (blockIdx.z % te) * kTile;
    const int rows = min(kChunk, a.T - n * kChunk);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const lm::bf16* k = a.x + (long long)n * kChunk * a.pitch + (size_t)a.H * a.D + (size_t)h * a.D + d0;
    const lm::bf16* v = a.x + (long long)n * kChunk * a.pitch + 2 * (size_t)a.H * a.D + (size_t)h * a.E + e0;
    lm::load_tile(vs, kLdT, v, a.pitch, kChunk, rows, min(kTile, a.E - e0), kTile, a.vec);
    const float* pw = a.decay_pow + (size_t)h * a.n_pow;
    const int kc = min(kTile, a.D - d0);
    constexpr int kVecs = kChunk * (kTile / 8) / 128;          // 16-byte pieces of the key tile per thread, all requested first
    __align__(16) lm::bf16 in[kVecs][8];
#pragma unroll
    for (int v = 0; v < kVecs; ++v) {
        const int i = threadIdx.x + v * 128, r = i / (kTile / 8), c = (i % (kTile / 8)) * 8;
        const lm::bf16* s = k + (long long)r * a.pitch + c;
        if (a.vec) *reinterpret_cast<uint4*>(in[v]) = r < rows && c < kc ? *reinterpret_cast<const uint4*>(s) : make_uint4(0u, 0u, 0u, 0u);
        else
#pragma unroll
            for (int e = 0; e < 8; ++e) in[v][e] = r < rows && c + e < kc ? s[e] : __float2bfloat16_rn(0.f);
    }
#pragma unroll
    for (int v = 0; v < kVecs; ++v) {
        const int i = threadIdx.x + v * 128, r = i / (kTile / 8), c = (i % (kTile / 8)) * 8;
        const float w = r < rows ? pw[rows - 1 - r] : 0.f;
        __align__(16) uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) lm::split2(w * __bfloat162float(in[v][2 * e]), w * __bfloat162float(in[v][2 * e + 1]), hi[e], lo[e]);
        *reinterpret_cast<uint4*>(kh + r * kLdT + c) = *reinterpret_cast<const uint4*>(hi);
        *reinterpret_cast<uint4*>(kl + r * kLdT + c) = *reinterpret_cast<const uint4*>(lo);
    }
    lm::cp_commit();
    lm::cp_wait<0>();
    __syncthreads();
    const int wd = (warp & 1) * 32, we = (warp >> 1) * 32;
    float acc[2][4][4] = {};
    for (int t0 = 0; t0 < rows; t0 += 16) {
        uint32_t ah[2][4], al[2][4], b[2][4];
#pragma unroll
        for (int m = 0; m < 2; ++m) {
            lm::load_a_t(ah[m], kh, kLdT, wd + 16 * m, t0);
            lm::load_a_t(al[m], kl, kLdT, wd + 16 * m, t0);
            lm::load_b_t(b[m], vs, kLdT, we + 16 * m, t0);
        }
#pragma unroll
        for (int m = 0; m < 2; ++m)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                lm::mma(acc[m][j], ah[m], b[j >> 1][(j & 1) * 2], b[j >> 1][(j & 1) * 2 + 1]);
                lm::mma(acc[m][j], al[m], b[j >> 1][(j & 1) * 2], b[j >> 1][(j & 1) * 2 + 1]);
            }
    }
    float* U = reinterpret_cast<float*>(a.scratch) + ((size_t)n * a.H + h) * a.D * a.E;
#pragma unroll
    for (int m = 0; m < 2; ++m)
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int q = 0; q < 4; q += 2) {
                const int d = d0 + wd + 16 * m + (lane >> 2) + (q >> 1) * 8, e = e0 + we + 8 * j + (lane & 3) * 2;
                if (d < a.D) store2(U + (size_t)d * a.E, e, a.E, acc[m][j][q], acc[m][j][q + 1]);
            }
}

// V neighbouring state elements of one head per thread
template <int V>
__global__ void __launch_bounds__(256) chunk_scan_kernel(const ChunkArgs a, int chunks) {
    rcu_kernel_entry();
    struct alignas(4 * V) Words { uint32_t w[V]; };
    struct alignas(4 * V) Floats { float f[V]; };
    const size_t per = (size_t)a.H * a.D * a.E / V, i = (size_t)blockIdx.x * 256 + threadIdx.x;
    if (i >= per) return;
    const float* pw = a.decay_pow + (i * V / ((size_t)a.D * a.E)) * a.n_pow;
    const float dc = pw[kChunk], dl = pw[a.T - (chunks - 1) * kChunk];
    Words* scratch = reinterpret_cast<Words*>(a.scratch) + i;
    Floats s = reinterpret_cast<const Floats*>(a.state)[i];
    constexpr int kAhead = 8;                  // chunks requested before the first of them is folded in
    for (int n0 = 0; n0 < chunks; n0 += kAhead) {
        Words u[kAhead];
#pragma unroll
        for (int j = 0; j < kAhead; ++j)
            if (n0 + j < chunks) u[j] = scratch[(size_t)(n0 + j) * per];
#pragma unroll
        for (int j = 0; j < kAhead; ++j) {
            if (n0 + j >= chunks) break;
            const float d = n0 + j == chunks - 1 ? dl : dc;
            Words o;
#pragma unroll
            for (int v = 0; v < V; ++v) {
                const lm::bf16 hi = __float2bfloat16_rn(s.f[v]);
                o.w[v] = lm::pack(__float2bfloat16_rn(s.f[v] - __bfloat162float(hi)), hi);
                s.f[v] = fmaf(d, s.f[v], __uint_as_float(u[j].w[v]));
            }
            scratch[(size_t)(n0 + j) * per] = o;
        }
    }
    reinterpret_cast<Floats*>(a.state)[i] = s;
}

__global__ void __launch_bounds__(256) chunk_out_kernel(const ChunkArgs a) {
    rcu_kernel_entry();
    extern __shared__ __align__(16) lm::bf16 tiles[];
    __shared__ float pw[kChunk + 1];
    const int dp = (a.D + 15) & ~15, ld = dp + 8;
    // the state's tiles, then - in the same place - the chunk's keys and values: two CTAs fit an SM
    lm::bf16 *qs = tiles, *sh = qs + kChunk * ld, *sl = sh + dp * kLdT, *ks = qs + kChunk * ld, *vs = ks + kChunk * ld;
    const int n = blockIdx.x, h = blockIdx.y, e0 = blockIdx.z * kTile;
    const int rows = min(kChunk, a.T - n * kChunk), ec = min(kTile, a.E - e0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const lm::bf16* q = a.x + (long long)n * kChunk * a.pitch + (size_t)h * a.D;
    lm::load_tile(qs, ld, q, a.pitch, kChunk, rows, a.D, dp, a.vec);
    lm::cp_commit();
    const uint32_t* S = a.scratch + ((size_t)n * a.H + h) * a.D * a.E + e0;
    if (a.E % 4 == 0) {
#pragma unroll 8
        for (int i = threadIdx.x; i < dp * (kTile / 4); i += 256) {
            const int d = i / (kTile / 4), c = (i % (kTile / 4)) * 4;
            const uint4 w = d < a.D && c < ec ? *reinterpret_cast<const uint4*>(S + (size_t)d * a.E + c) : make_uint4(0u, 0u, 0u, 0u);
            *reinterpret_cast<uint2*>(sh + d * kLdT + c) = make_uint2((w.x >> 16) | (w.y & 0xffff0000u), (w.z >> 16) | (w.w & 0xffff0000u));
            *reinterpret_cast<uint2*>(sl + d * kLdT + c) = make_uint2((w.x & 0xffffu) | (w.y << 16), (w.z & 0xffffu) | (w.w << 16));
        }
    } else {
        for (int i = threadIdx.x; i < dp * kTile; i += 256) {
            const int d = i / kTile, c = i % kTile;
            const uint32_t w = d < a.D && c < ec ? S[(size_t)d * a.E + c] : 0u;
            sh[d * kLdT + c] = __ushort_as_bfloat16((unsigned short)(w >> 16));
            sl[d * kLdT + c] = __ushort_as_bfloat16((unsigned short)w);
        }
    }
    for (int i = threadIdx.x; i <= kChunk; i += 256) pw[i] = a.decay_pow[(size_t)h * a.n_pow + i];
    lm::cp_wait<0>();
    __syncthreads();
    const int r0 = warp * 16;
    float o[8][4] = {};
    // what the tokens before the chunk left in the state
    for (int k0 = 0; k0 < dp && r0 < rows; k0 += 16) {
        uint32_t qa[4];
        lm::load_a(qa, qs, ld, r0, k0);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            uint32_t bh[4], bl[4];
            lm::load_b_t(bh, sh, kLdT, 16 * j, k0);
            lm::load_b_t(bl, sl, kLdT, 16 * j, k0);
            lm::mma(o[2 * j], qa, bh[0], bh[1]);
            lm::mma(o[2 * j + 1], qa, bh[2], bh[3]);
            lm::mma(o[2 * j], qa, bl[0], bl[1]);
            lm::mma(o[2 * j + 1], qa, bl[2], bl[3]);
        }
    }
    __syncthreads();
    lm::load_tile(ks, ld, q + (size_t)a.H * a.D, a.pitch, kChunk, rows, a.D, dp, a.vec);
    lm::load_tile(vs, kLdT, a.x + (long long)n * kChunk * a.pitch + 2 * (size_t)a.H * a.D + (size_t)h * a.E + e0, a.pitch, kChunk, rows, ec, kTile, a.vec);
    lm::cp_commit();
    lm::cp_wait<0>();
    __syncthreads();
    if (r0 >= rows) return;
    const int i0 = r0 + g, i1 = i0 + 8;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
        o[j][0] *= pw[i0 + 1]; o[j][1] *= pw[i0 + 1];
        o[j][2] *= pw[i1 + 1]; o[j][3] *= pw[i1 + 1];
    }
    // the chunk's own tokens, 32 keys at a time up to this warp's rows
    for (int j0 = 0; j0 <= r0; j0 += 32) {
        float s[4][4] = {};
        for (int k0 = 0; k0 < dp; k0 += 16) {
            uint32_t qa[4], b0[4], b1[4];
            lm::load_a(qa, qs, ld, r0, k0);
            lm::load_b(b0, ks, ld, j0, k0);
            lm::load_b(b1, ks, ld, j0 + 16, k0);
            lm::mma(s[0], qa, b0[0], b0[1]);
            lm::mma(s[1], qa, b0[2], b0[3]);
            lm::mma(s[2], qa, b1[0], b1[1]);
            lm::mma(s[3], qa, b1[2], b1[3]);
        }
#pragma unroll
        for (int c = 0; c < 4; ++c)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int i = e < 2 ? i0 : i1, j = j0 + 8 * c + 2 * t + (e & 1);
                s[c][e] = j <= i ? s[c][e] * pw[i - j] : 0.f;
            }
#pragma unroll
        for (int kk = 0; kk < 2; ++kk) {
            uint32_t ph[4], pl[4];
            lm::split2(s[2 * kk][0], s[2 * kk][1], ph[0], pl[0]);
            lm::split2(s[2 * kk][2], s[2 * kk][3], ph[1], pl[1]);
            lm::split2(s[2 * kk + 1][0], s[2 * kk + 1][1], ph[2], pl[2]);
            lm::split2(s[2 * kk + 1][2], s[2 * kk + 1][3], ph[3], pl[3]);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                uint32_t b[4];
                lm::load_b_t(b, vs, kLdT, 16 * j, j0 + 16 * kk);
                lm::mma(o[2 * j], ph, b[0], b[1]);
                lm::mma(o[2 * j + 1], ph, b[2], b[3]);
                lm::mma(o[2 * j], pl, b[0], b[1]);
                lm::mma(o[2 * j + 1], pl, b[2], b[3]);
            }
        }
    }
    float* out = a.out + (size_t)n * kChunk * a.H * a.E + (size_t)h * a.E + e0;
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
            const int i = e < 2 ? i0 : i1, c = 8 * j + 2 * t;
            if (i >= rows) continue;
            float* row = out + (size_t)i * a.H * a.E;
            if (a.E % 2 == 0) {
                store2(row, c, ec, o[j][e], o[j][e + 1]);
            } else {
                if (c < ec) row[c] = o[j][e];
                if (c + 1 < ec) row[c + 1] = o[j][e + 1];
            }
        }
}

size_t chunk_out_smem(int D) {
    const size_t dp = (D + 15) & ~15;
    return (kChunk * (dp + 8) + std::max(kChunk * (dp + 8) + kChunk * kLdT, 2 * dp * kLdT)) * sizeof(lm::bf16);
}

rcu_status launch_chunks(rcu_device* dev, const LightningArgs& l) {
    const int chunks = (l.T + kChunk - 1) / kChunk;
    void* scratch = nullptr;
    rcu_status st = rcu_alloc(dev, (uint64_t)chunks * l.H * l.D * l.E * 4, &scratch);
    if (st != RCU_OK) return st;
    ChunkArgs a{(const lm::bf16*)l.x, l.pitch, l.decay_pow, l.n_pow, l.state, (uint32_t*)scratch, l.out, l.T, l.H, l.D, l.E, 0};
    a.vec = l.D % 8 == 0 && l.E % 8 == 0 && l.pitch % 8 == 0 && (reinterpret_cast<uintptr_t>(l.x) & 15) == 0;
    const int td = (l.D + kTile - 1) / kTile, te = (l.E + kTile - 1) / kTile;
    const size_t smem_kv = 3 * (size_t)kChunk * kLdT * sizeof(lm::bf16), smem_out = chunk_out_smem(l.D);
    RCU_CUDA(dev, cudaFuncSetAttribute(chunk_kv_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_kv));
    RCU_CUDA(dev, cudaFuncSetAttribute(chunk_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_out));
    rcu_launch(dev, chunk_kv_kernel, dim3(chunks, l.H, td * te), 128, smem_kv, a);
    const size_t elems = (size_t)l.H * l.D * l.E;
    if ((size_t)l.D * l.E % 4 == 0 && (reinterpret_cast<uintptr_t>(l.state) & 15) == 0)
        rcu_launch(dev, chunk_scan_kernel<4>, (unsigned)((elems / 4 + 255) / 256), 256, 0, a, chunks);
    else rcu_launch(dev, chunk_scan_kernel<1>, (unsigned)((elems + 255) / 256), 256, 0, a, chunks);
    rcu_launch(dev, chunk_out_kernel, dim3(chunks, l.H, te), 256, smem_out, a);
    rcu_free(dev, scratch);                    // the pool reuses blocks in stream order
    dev->launches += 2;
    RCU_LAUNCH_CHECK(dev);
    return RCU_OK;
}

}  // namespace

extern "C" rcu_status rcu_lightning(rcu_device* dev, const rcu_tensor* x, const rcu_tensor* decay_pow, rcu_tensor* state, rcu_tensor* dst) {
    if (!dev) return RCU_ERR_INVALID_ARG;
    RCU_REQUIRE(dev, t_valid(x) && t_valid(decay_pow) && t_valid(state) && t_valid(dst), "lightning: invalid tensor descriptor");
    RCU_REQUIRE(dev, x->dt == RCU_F32 || x->dt == RCU_BF16, "lightning: f32 or bf16 rows");
    RCU_REQUIRE(dev, state->dt == RCU_F32 && state->rank == 3 && dst->dt == RCU_F32, "lightning: the state is f32 [heads, dim, vdim], the output f32");
    const uint64_t H = state->shape[0], D = state->shape[1], E = state->shape[2];
    const uint64_t pitch = x->shape[x->rank - 1], T = t_numel(x) / pitch;
    RCU_REQUIRE(dev, decay_pow->dt == RCU_F32 && decay_pow->rank == 2 && decay_pow->shape[0] == H && decay_pow->shape[1] >= 2,
                "lightning: decay powers are f32 [heads, >= 2]");
    RCU_REQUIRE(dev, 2 * H * D + H * E <= pitch && t_numel(dst) == T * H * E, "lightning: rows or output do not fit heads x (dim, dim, vdim)");
    if (D > 512 || H > 65535 || E > 65535 * 32ull || T > 0x7fffffffull) return rcu_fail(dev, RCU_ERR_UNSUPPORTED, "lightning: dim %llu (at most 512)", (unsigned long long)D);
    DevGuard g(dev->ordinal);
    LightningArgs a{x->data, (long long)pitch, (const float*)decay_pow->data, (int)decay_pow->shape[1], (float*)state->data, (float*)dst->data,
                    (int)T, (int)H, (int)D, (int)E};
    if (x->dt == RCU_BF16 && T > 32 && a.n_pow > kChunk && chunk_out_smem(a.D) + 1024 <= (size_t)dev->smem_optin) return launch_chunks(dev, a);
    return x->dt == RCU_F32 ? launch_recurrent<float>(dev, a) : launch_recurrent<__nv_bfloat16>(dev, a);
}
