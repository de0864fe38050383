// Attention of one decoded token over a layer's ring of keys and values (grouped_attention.cu describes the cache): part of the
// fused decode step (stack_decode.cu).
//
// The visible positions are cut into tiles of 16 that CTAs and warps take in turn.  Every CTA norms and rotates the queries of its
// heads; the one whose tile holds the current position first norms, rotates and stores the token's key and its value.  The partial
// results of a kv head's CTAs (maximum, sum of weights, weighted values) are merged, and the sink added, through distributed shared
// memory when the CTAs form one cluster of up to eight; more of them leave their parts in global memory, where the last to finish
// merges them.
//   grouped_step_mma_kernel   bf16 rings on the tensor cores: up to 16 query heads of a kv head against 16 positions, operands
//                             straight from global memory in registers, queries and weights as bf16 value plus remainder;
//   grouped_step_kernel       any type and size in FFMA.
#pragma once
#include <cooperative_groups.h>

#include <algorithm>

#include "lm_mma.cuh"
#include "window.cuh"

namespace gstep {

constexpr int kThreads = 256, kWarps = 8;
constexpr int kTile = 16;             // positions per tile
constexpr int kMmaHeads = 16;         // query heads per CTA of the tensor-core kernel
constexpr int kFmaHeads = 8;          // of the other (one warp each)
constexpr int kMaxSplits = 64;
constexpr int kCluster = 8;           // CTAs of a kv head that merge through distributed shared memory

struct Args {
    const float* mix;                 // the token's query heads [H, D], key heads [G, D], value heads [G, E]
    const float *q_scale, *k_scale;   // [D]
    const float2* angles;             // (cos, sin) of the current position's pairs
    const float* sink;                // [H], nullable
    void* ring;                       // [ring_rows, G * (D + E)]
    const uint32_t* d_pos;
    float* out;                       // [H, E]
    float* partial;                   // [splits][H][pitch]: E sums, the maximum, the sum of the weights
    uint32_t* arrived;                // one counter per blockIdx.y, zero between steps
    int H, G, D, E, pairs, ring_rows, window, chunk;
    float eps, scale;
};

__host__ __device__ __forceinline__ int pitch_of(int E) { return ((E + 3) & ~3) + 4; }
__host__ __device__ __forceinline__ int head_groups(int H, int G, int per) { return (H / G + per - 1) / per; }

// One head of the current token, normed and rotated, by a warp: put(d, value)
template <class Put> __device__ __forceinline__ void current_head(const Args& a, const float* x, const float* scale, Put put) {
    const int lane = threadIdx.x & 31;
    float q = 0.f;
    for (int d = lane; d < a.D; d += 32) q = fmaf(x[d], x[d], q);
    const float rstd = 1.0f / sqrtf(warp_sum(q) / (float)a.D + a.eps);
    for (int i = lane; 2 * i < a.D; i += 32) {
        const int d = 2 * i;
        const float u = x[d] * rstd * scale[d], v = d + 1 < a.D ? x[d + 1] * rstd * scale[d + 1] : 0.f;
        if (i < a.pairs) {
            const float2 cs = a.angles[i];
            put(d, u * cs.x - v * cs.y);
            put(d + 1, v * cs.x + u * cs.y);
        } else {
            put(d, u);
            if (d + 1 < a.D) put(d + 1, v);
        }
    }
}

// The current token's key and value of kv head g into its ring row (by one warp); the CTA sees them after a barrier.
template <class T> __device__ __forceinline__ void append(const Args& a, int g, uint32_t pos) {
    T* row = reinterpret_cast<T*>(a.ring) + (size_t)(pos % (uint32_t)a.ring_rows) * a.G * (a.D + a.E);
    T *k = row + (size_t)g * a.D, *v = row + (size_t)a.G * a.D + (size_t)g * a.E;
    current_head(a, a.mix + (size_t)(a.H + g) * a.D, a.k_scale, [&](int d, float x) { k[d] = from_f32<T>(x); });
    const float* xv = a.mix + (size_t)(a.H + a.G) * a.D + (size_t)g * a.E;
    for (int e = threadIdx.x & 31; e < a.E; e += 32) v[e] = from_f32<T>(xv[e]);
}

// What every CTA does once its partial results are written: the last of the `active` CTAs of this blockIdx.y merges heads [h0, h0 + nh).
__device__ __forceinline__ void merge(const Args& a, int h0, int nh, int active, float* weights /* [kMaxSplits + 1][16] */) {
    __shared__ int last;
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) {
        last = atomicAdd(&a.arrived[blockIdx.y], 1u) == (uint32_t)active - 1;
        if (last) a.arrived[blockIdx.y] = 0;
    }
    __syncthreads();
    if (!last) return;
    __threadfence();
    const int pitch = pitch_of(a.E), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const size_t stride = (size_t)a.H * pitch;
    const float* base = a.partial + (size_t)h0 * pitch;
    for (int h = warp; h < nh; h += kWarps) {
        const float* p = base + (size_t)h * pitch + pitch - 2;
        float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
        if (lane < active) { m0 = __ldcg(p + lane * stride); l0 = __ldcg(p + lane * stride + 1); }
        if (lane + 32 < active) { m1 = __ldcg(p + (lane + 32) * stride); l1 = __ldcg(p + (lane + 32) * stride + 1); }
        const float M = warp_max(fmaxf(m0, m1));
        const float w0 = lane < active ? expf(m0 - M) : 0.f, w1 = lane + 32 < active ? expf(m1 - M) : 0.f;
        float l = warp_sum(w0 * l0 + w1 * l1);
        if (a.sink) l += expf(a.sink[h0 + h] - M);
        weights[lane * 16 + h] = w0 / l;
        weights[(lane + 32) * 16 + h] = w1 / l;
    }
    __syncthreads();
    const int quads = (a.E + 3) / 4;
    for (int i = threadIdx.x; i < nh * quads; i += kThreads) {
        const int h = i / quads, e = (i - h * quads) * 4;
        const float* p = base + (size_t)h * pitch + e;
        float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
        for (int j = 0; j < active; ++j) {
            const float4 v = __ldcg(reinterpret_cast<const float4*>(p + j * stride));
            const float w = weights[j * 16 + h];
            s.x = fmaf(w, v.x, s.x);
            s.y = fmaf(w, v.y, s.y);
            s.z = fmaf(w, v.z, s.z);
            s.w = fmaf(w, v.w, s.w);
        }
        float* o = a.out + (size_t)(h0 + h) * a.E + e;
        o[0] = s.x;
        if (e + 1 < a.E) o[1] = s.y;
        if (e + 2 < a.E) o[2] = s.z;
        if (e + 3 < a.E) o[3] = s.w;
    }
}

// NB: blocks of 32 key features, EB: blocks of 64 value features (D and E multiples of 8).  The products' inner index may run over the
// features in any order as long as both operands agree: a lane takes eight consecutive features of a key row in one load and feeds
// them to two products; value columns are dealt to the product's columns eight apart in the same way.  CL: the CTAs of blockIdx.y are
// one cluster.
template <int NB, int EB, bool CL>
__global__ void __launch_bounds__(kThreads) grouped_step_mma_kernel(const Args a) {
    using lm::bf16;
    extern __shared__ __align__(16) unsigned char smem[];
    constexpr int ldq = NB * 32 + 8, KP = NB / 2;                         // KP: pairs of features per lane
    bf16 *qh = reinterpret_cast<bf16*>(smem), *ql = qh + kMmaHeads * ldq;
    float* acc_s = reinterpret_cast<float*>(ql + kMmaHeads * ldq);        // [warps][nh][E]; the CTA's sums end up in the first [nh][E]
    __shared__ float m_s[kWarps][kMmaHeads], l_s[kWarps][kMmaHeads], weights[kMaxSplits * 16];
    __shared__ float cta_m[kMmaHeads], cta_l[kMmaHeads];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, gr = lane >> 2, t = lane & 3;
    const int per = a.H / a.G, groups = head_groups(a.H, a.G, kMmaHeads);
    const int g = blockIdx.y / groups, hg = (blockIdx.y - g * groups) * kMmaHeads;
    const int h0 = g * per + hg, nh = min(kMmaHeads, per - hg);
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    // constants first: the norms' scales, and zeros for what no head fills
    float2 qs[KP], ks[KP];
#pragma unroll
    for (int i = 0; i < KP; ++i) {
        const int d = 2 * (lane + 32 * i);
        qs[i] = d < a.D ? *reinterpret_cast<const float2*>(a.q_scale + d) : make_float2(0.f, 0.f);
        ks[i] = d < a.D ? *reinterpret_cast<const float2*>(a.k_scale + d) : make_float2(0.f, 0.f);
    }
    for (int h = warp; h < kMmaHeads; h += kWarps)
        for (int d = lane; d < ldq; d += 32)
            if (h >= nh || d >= a.D) qh[h * ldq + d] = ql[h * ldq + d] = __float2bfloat16_rn(0.f);
    asm volatile("griddepcontrol.wait;" ::: "memory");

    const uint32_t pos = *a.d_pos;
    // the token's heads this warp prepares (two query heads; the last warp also the key and the value) and the angles, all in flight at once
    float2 xq[2][KP], xk[KP], cs[KP];
    const float* key = a.mix + (size_t)(a.H + g) * a.D;
#pragma unroll
    for (int i = 0; i < KP; ++i) {
        const int d = 2 * (lane + 32 * i);
        cs[i] = lane + 32 * i < a.pairs ? a.angles[lane + 32 * i] : make_float2(1.f, 0.f);
#pragma unroll
        for (int x = 0; x < 2; ++x)
            xq[x][i] = d < a.D && warp + x * kWarps < nh ? *reinterpret_cast<const float2*>(a.mix + (size_t)(h0 + warp + x * kWarps) * a.D + d) : make_float2(0.f, 0.f);
        xk[i] = d < a.D && warp == kWarps - 1 ? *reinterpret_cast<const float2*>(key + d) : make_float2(0.f, 0.f);
    }
    const Visible see{a.window, a.chunk, 0};
    const int low = see.first((int)pos), n = (int)pos - low + 1, tiles = (n + kTile - 1) / kTile;
    const int active = min((int)gridDim.x, tiles);
    if (!CL && (int)blockIdx.x >= active) return;

    const size_t W = (size_t)a.G * (a.D + a.E);
    const bf16* K = reinterpret_cast<const bf16*>(a.ring) + (size_t)g * a.D;
    const bf16* V = reinterpret_cast<const bf16*>(a.ring) + (size_t)a.G * a.D + (size_t)g * a.E;
    uint4 k[NB][2], v[EB][4];
    auto load = [&](int p0) {
        const int base = p0 % a.ring_rows;
        auto row = [&](int i) {               // positions beyond the current one: any row, weight zero
            const int r = base + min(i, (int)pos - p0);
            return (size_t)(r < a.ring_rows ? r : r - a.ring_rows) * W;
        };
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const bf16* src = K + row(i * 8 + gr);
#pragma unroll
            for (int b = 0; b < NB; ++b) {
                const int d = b * 32 + t * 8;
                k[b][i] = d < a.D ? *reinterpret_cast<const uint4*>(src + d) : make_uint4(0u, 0u, 0u, 0u);
            }
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const bf16* src = V + row((i >> 1) * 8 + 2 * t + (i & 1));
#pragma unroll
            for (int c = 0; c < EB; ++c) {
                const int e = c * 64 + gr * 8;
                v[c][i] = e < a.E ? *reinterpret_cast<const uint4*>(src + e) : make_uint4(0u, 0u, 0u, 0u);
            }
        }
    };
    const int first = (int)blockIdx.x + warp * active, step = active * kWarps;
    const bool mine = (int)blockIdx.x < active && first < tiles, early = mine && low + first * kTile + kTile <= (int)pos;
    if (early) load(low + first * kTile);     // cached rows only: they travel while the queries are prepared

    // norm and rotation of a head in registers
    auto prepare = [&](float2(&x)[KP], const float2(&scale)[KP]) {
        float q = 0.f;
#pragma unroll
        for (int i = 0; i < KP; ++i) q += x[i].x * x[i].x + x[i].y * x[i].y;
        const float rstd = 1.0f / sqrtf(warp_sum(q) / (float)a.D + a.eps);
#pragma unroll
        for (int i = 0; i < KP; ++i) {
            const float u = x[i].x * rstd * scale[i].x, w = x[i].y * rstd * scale[i].y;
            x[i] = make_float2(u * cs[i].x - w * cs[i].y, w * cs[i].x + u * cs[i].y);
        }
    };
#pragma unroll
    for (int x = 0; x < 2; ++x) {
        const int h = warp + x * kWarps;
        if (h >= nh) break;
        prepare(xq[x], qs);
#pragma unroll
        for (int i = 0; i < KP; ++i) {
            const int d = 2 * (lane + 32 * i);
            uint32_t hi, lo;
            lm::split2(xq[x][i].x * a.scale, xq[x][i].y * a.scale, hi, lo);
            if (d < a.D) {
                *reinterpret_cast<uint32_t*>(qh + h * ldq + d) = hi;
                *reinterpret_cast<uint32_t*>(ql + h * ldq + d) = lo;
            }
        }
    }
    if (warp == kWarps - 1 && (tiles - 1) % active == (int)blockIdx.x) {
        bf16* dst = reinterpret_cast<bf16*>(a.ring) + (size_t)(pos % (uint32_t)a.ring_rows) * W;
        prepare(xk, ks);
#pragma unroll
        for (int i = 0; i < KP; ++i) {
            const int d = 2 * (lane + 32 * i);
            if (d < a.D) *reinterpret_cast<__nv_bfloat162*>(dst + (size_t)g * a.D + d) = __floats2bfloat162_rn(xk[i].x, xk[i].y);
        }
        const float* xv = a.mix + (size_t)(a.H + a.G) * a.D + (size_t)g * a.E;
        for (int e = 2 * lane; e < a.E; e += 64) {
            const float2 u = *reinterpret_cast<const float2*>(xv + e);
            *reinterpret_cast<__nv_bfloat162*>(dst + (size_t)a.G * a.D + (size_t)g * a.E + e) = __floats2bfloat162_rn(u.x, u.y);
        }
    }
    __syncthreads();

    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f, o[EB][8][4];
#pragma unroll
    for (int c = 0; c < EB; ++c)
#pragma unroll
        for (int j = 0; j < 8; ++j) o[c][j][0] = o[c][j][1] = o[c][j][2] = o[c][j][3] = 0.f;
    for (int tile = mine ? first : tiles; tile < tiles; tile += step) {
        const int p0 = low + tile * kTile;
        if (tile != first || !early) load(p0);
        float s0[4] = {}, s1[4] = {};
#pragma unroll
        for (int b = 0; b < NB; ++b)
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                const int d = b * 32 + t * 8 + x * 4;
                const uint2 h_lo = *reinterpret_cast<const uint2*>(qh + gr * ldq + d), h_hi = *reinterpret_cast<const uint2*>(qh + (gr + 8) * ldq + d);
                const uint2 r_lo = *reinterpret_cast<const uint2*>(ql + gr * ldq + d), r_hi = *reinterpret_cast<const uint2*>(ql + (gr + 8) * ldq + d);
                const uint32_t ah[4] = {h_lo.x, h_hi.x, h_lo.y, h_hi.y}, al[4] = {r_lo.x, r_hi.x, r_lo.y, r_hi.y};
                const uint32_t k0a = x ? k[b][0].z : k[b][0].x, k0b = x ? k[b][0].w : k[b][0].y;
                const uint32_t k1a = x ? k[b][1].z : k[b][1].x, k1b = x ? k[b][1].w : k[b][1].y;
                lm::mma(s0, ah, k0a, k0b);
                lm::mma(s1, ah, k1a, k1b);
                lm::mma(s0, al, k0a, k0b);
                lm::mma(s1, al, k1a, k1b);
            }
        // rows gr and gr + 8 are heads; columns 2 t, 2 t + 1 (s0) and 8 + 2 t, 9 + 2 t (s1) positions
        float t0 = -INFINITY, t1 = -INFINITY;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            if (p0 + 2 * t + (e & 1) > (int)pos) s0[e] = -INFINITY;
            if (p0 + 8 + 2 * t + (e & 1) > (int)pos) s1[e] = -INFINITY;
            if (e < 2) t0 = fmaxf(t0, fmaxf(s0[e], s1[e]));
            else t1 = fmaxf(t1, fmaxf(s0[e], s1[e]));
        }
#pragma unroll
        for (int x = 1; x < 4; x *= 2) {
            t0 = fmaxf(t0, __shfl_xor_sync(0xffffffffu, t0, x));
            t1 = fmaxf(t1, __shfl_xor_sync(0xffffffffu, t1, x));
        }
        const float n0 = fmaxf(m0, t0), n1 = fmaxf(m1, t1), c0 = expf(m0 - n0), c1 = expf(m1 - n1);       // a tile holds at least one position
        m0 = n0; m1 = n1;
        l0 *= c0; l1 *= c1;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            s0[e] = expf(s0[e] - (e < 2 ? m0 : m1));
            s1[e] = expf(s1[e] - (e < 2 ? m0 : m1));
            if (e < 2) l0 += s0[e] + s1[e];
            else l1 += s0[e] + s1[e];
        }
        uint32_t ph[4], pl[4];
        lm::split2(s0[0], s0[1], ph[0], pl[0]);
        lm::split2(s0[2], s0[3], ph[1], pl[1]);
        lm::split2(s1[0], s1[1], ph[2], pl[2]);
        lm::split2(s1[2], s1[3], ph[3], pl[3]);
#pragma unroll
        for (int c = 0; c < EB; ++c) {
            const uint32_t w[4][4] = {{v[c][0].x, v[c][0].y, v[c][0].z, v[c][0].w}, {v[c][1].x, v[c][1].y, v[c][1].z, v[c][1].w},
                                      {v[c][2].x, v[c][2].y, v[c][2].z, v[c][2].w}, {v[c][3].x, v[c][3].y, v[c][3].z, v[c][3].w}};
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                const uint32_t sel = j & 1 ? 0x7632u : 0x5410u;
                const uint32_t b0 = __byte_perm(w[0][j >> 1], w[1][j >> 1], sel), b1 = __byte_perm(w[2][j >> 1], w[3][j >> 1], sel);
                float(&oc)[4] = o[c][j];
                oc[0] *= c0; oc[1] *= c0; oc[2] *= c1; oc[3] *= c1;
                lm::mma(oc, ph, b0, b1);
                lm::mma(oc, pl, b0, b1);
            }
        }
    }
#pragma unroll
    for (int x = 1; x < 4; x *= 2) {
        l0 += __shfl_xor_sync(0xffffffffu, l0, x);
        l1 += __shfl_xor_sync(0xffffffffu, l1, x);
    }
    if (t == 0) {
        m_s[warp][gr] = m0; m_s[warp][gr + 8] = m1;
        l_s[warp][gr] = l0; l_s[warp][gr + 8] = l1;
    }
    // column 2 t + (e & 1) of product j is value feature c * 64 + 8 (2 t + (e & 1)) + j
    if (mine)
#pragma unroll
        for (int c = 0; c < EB; ++c)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int h = gr + (e >> 1) * 8, col = c * 64 + (2 * t + (e & 1)) * 8;
                if (h < nh && col < a.E) {
                    float4* dst = reinterpret_cast<float4*>(acc_s + ((size_t)warp * nh + h) * a.E + col);
                    dst[0] = make_float4(o[c][0][e], o[c][1][e], o[c][2][e], o[c][3][e]);
                    dst[1] = make_float4(o[c][4][e], o[c][5][e], o[c][6][e], o[c][7][e]);
                }
            }
    __syncthreads();
    // the warps' parts of a head, four features per thread; a warp without a tile has the maximum -inf and left no sums
    const int quads = a.E / 4;
    const int pitch = pitch_of(a.E);
    float* part = CL ? acc_s : a.partial + ((size_t)blockIdx.x * a.H + h0) * pitch;
    for (int i = threadIdx.x; i < nh * quads; i += kThreads) {
        const int h = i / quads, e = (i - h * quads) * 4;
        float M = -INFINITY, l = 0.f;
        float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int w = 0; w < kWarps; ++w) M = fmaxf(M, m_s[w][h]);
#pragma unroll
        for (int w = 0; w < kWarps; ++w) {
            if (m_s[w][h] == -INFINITY) continue;
            const float f = expf(m_s[w][h] - M);
            const float4 x = *reinterpret_cast<const float4*>(acc_s + ((size_t)w * nh + h) * a.E + e);
            s.x = fmaf(f, x.x, s.x);
            s.y = fmaf(f, x.y, s.y);
            s.z = fmaf(f, x.z, s.z);
            s.w = fmaf(f, x.w, s.w);
            l = fmaf(f, l_s[w][h], l);
        }
        *reinterpret_cast<float4*>(part + (CL ? (size_t)h * a.E : (size_t)h * pitch) + e) = s;      // CL: over warp 0's part, read by this thread only
        if (e == 0) {
            if (CL) {
                cta_m[h] = M;
                cta_l[h] = l;
            } else {
                part[(size_t)h * pitch + pitch - 2] = M;
                part[(size_t)h * pitch + pitch - 1] = l;
            }
        }
    }
    if (!CL) {
        merge(a, h0, nh, active, weights);
        return;
    }
    namespace cg = cooperative_groups;
    cg::cluster_group cluster = cg::this_cluster();
    cluster.sync();
    // every CTA merges a share of the outputs
    for (int i = (int)blockIdx.x * kThreads + threadIdx.x; i < nh * quads; i += (int)gridDim.x * kThreads) {
        const int h = i / quads, e = (i - h * quads) * 4;
        float M = -INFINITY, ms[kCluster], ls[kCluster];
        float4 x[kCluster];
#pragma unroll
        for (int j = 0; j < kCluster; ++j)
            if (j < active) {
                ms[j] = *cluster.map_shared_rank(&cta_m[h], j);
                ls[j] = *cluster.map_shared_rank(&cta_l[h], j);
                x[j] = *reinterpret_cast<const float4*>(cluster.map_shared_rank(acc_s + (size_t)h * a.E + e, j));
            }
#pragma unroll
        for (int j = 0; j < kCluster; ++j)
            if (j < active) M = fmaxf(M, ms[j]);
        float l = a.sink ? expf(a.sink[h0 + h] - M) : 0.f;
        float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int j = 0; j < kCluster; ++j)
            if (j < active) {
                const float f = expf(ms[j] - M);
                l = fmaf(f, ls[j], l);
                s.x = fmaf(f, x[j].x, s.x);
                s.y = fmaf(f, x[j].y, s.y);
                s.z = fmaf(f, x[j].z, s.z);
                s.w = fmaf(f, x[j].w, s.w);
            }
        const float inv = 1.0f / l;
        *reinterpret_cast<float4*>(a.out + (size_t)(h0 + h) * a.E + e) = make_float4(s.x * inv, s.y * inv, s.z * inv, s.w * inv);
    }
    cluster.sync();                       // no CTA leaves while its shared memory is being read
}

// A warp per head; tiles of positions staged in shared memory and shared by the heads; a lane owns every 32nd feature.
template <class T, int PE>
__global__ void __launch_bounds__(kThreads) grouped_step_kernel(const Args a) {
    rcu_kernel_entry();
    extern __shared__ __align__(16) unsigned char smem[];
    float* q_s = reinterpret_cast<float*>(smem);                          // [kFmaHeads][D]
    T* rows = reinterpret_cast<T*>(q_s + (size_t)kFmaHeads * a.D);         // [kTile][D + E]
    __shared__ float weights[kMaxSplits * 16];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int per = a.H / a.G, groups = head_groups(a.H, a.G, kFmaHeads);
    const int g = blockIdx.y / groups, hg = (blockIdx.y - g * groups) * kFmaHeads;
    const int h0 = g * per + hg, nh = min(kFmaHeads, per - hg);
    const uint32_t pos = *a.d_pos;
    const Visible see{a.window, a.chunk, 0};
    const int low = see.first((int)pos), n = (int)pos - low + 1, tiles = (n + kTile - 1) / kTile;
    const int active = min((int)gridDim.x, tiles);
    if ((int)blockIdx.x >= active) return;
    float* q = q_s + (size_t)warp * a.D;
    if (warp < nh) current_head(a, a.mix + (size_t)(h0 + warp) * a.D, a.q_scale, [&](int d, float v) { q[d] = v; });
    if ((tiles - 1) % active == (int)blockIdx.x && warp == kWarps - 1) append<T>(a, g, pos);
    const int W1 = a.D + a.E;
    const size_t W = (size_t)a.G * W1;
    const T* ring = reinterpret_cast<const T*>(a.ring);
    float m = -INFINITY, l = 0.f, o[PE];
#pragma unroll
    for (int c = 0; c < PE; ++c) o[c] = 0.f;
    for (int tile = blockIdx.x; tile < tiles; tile += active) {
        const int p0 = low + tile * kTile, np = min(kTile, (int)pos + 1 - p0);
        __syncthreads();
        for (int r = warp; r < np; r += kWarps) {
            const T* src = ring + (size_t)((p0 + r) % a.ring_rows) * W;
            T* dst = rows + (size_t)r * W1;
            for (int d = lane; d < a.D; d += 32) dst[d] = src[(size_t)g * a.D + d];
            for (int e = lane; e < a.E; e += 32) dst[a.D + e] = src[(size_t)a.G * a.D + (size_t)g * a.E + e];
        }
        __syncthreads();
        if (warp >= nh) continue;
        float s[kTile], top = -INFINITY;
#pragma unroll
        for (int r = 0; r < kTile; ++r) {
            s[r] = 0.f;
            if (r < np)
                for (int d = lane; d < a.D; d += 32) s[r] = fmaf(q[d], to_f32<T>(rows[(size_t)r * W1 + d]), s[r]);
        }
#pragma unroll
        for (int r = 0; r < kTile; ++r) {
            s[r] = r < np ? warp_sum(s[r]) * a.scale : -INFINITY;
            top = fmaxf(top, s[r]);
        }
        const float mn = fmaxf(m, top), corr = expf(m - mn);
        m = mn;
        l *= corr;
#pragma unroll
        for (int c = 0; c < PE; ++c) o[c] *= corr;
#pragma unroll
        for (int r = 0; r < kTile; ++r) {
            if (r >= np) break;
            const float p = expf(s[r] - m);
            l += p;
            const T* v = rows + (size_t)r * W1 + a.D;
#pragma unroll
            for (int c = 0; c < PE; ++c)
                if (lane + 32 * c < a.E) o[c] = fmaf(p, to_f32<T>(v[lane + 32 * c]), o[c]);
        }
    }
    if (warp < nh) {
        const int pitch = pitch_of(a.E);
        float* part = a.partial + ((size_t)blockIdx.x * a.H + h0 + warp) * pitch;
#pragma unroll
        for (int c = 0; c < PE; ++c)
            if (lane + 32 * c < a.E) part[lane + 32 * c] = o[c];
        if (lane == 0) {
            part[pitch - 2] = m;
            part[pitch - 1] = l;
        }
    }
    merge(a, h0, nh, active, weights);
}

inline bool takes_mma(int dt, int D, int E, const void* ring) {
    return dt == RCU_BF16 && D % 8 == 0 && E % 8 == 0 && D <= 256 && E <= 256 && (reinterpret_cast<uintptr_t>(ring) & 15) == 0;
}

// CTAs (grid.x) of a layer whose tokens see at most `most` rows: one tile per warp, as far as a cluster goes (`clusters`), beyond that
// as many as the device holds
inline int splits(int sm_count, int rows_y, uint64_t most, bool clusters) {
    const int tiles = (int)std::min<uint64_t>((most + kTile - 1) / kTile, 1u << 26), want = (tiles + kWarps - 1) / kWarps;
    if (clusters && want <= 4 * kCluster) return std::min(kCluster, std::max(1, (tiles + 1) / 2));
    const int room = std::max(1, 2 * sm_count / std::max(1, rows_y));
    return std::max(1, std::min(std::min(kMaxSplits, room), want));
}

inline rcu_status launch(rcu_device* dev, int dt, const Args& a, int n_splits) {
    const bool mma = takes_mma(dt, a.D, a.E, a.ring);
    const int heads = mma ? kMmaHeads : kFmaHeads, nh = a.H / a.G < heads ? a.H / a.G : heads;
    const dim3 grid(n_splits, a.G * head_groups(a.H, a.G, heads));
    const bool cluster = mma && n_splits <= kCluster;
#define RCU_GS(KERN_)                                                                                                            \
    do {                                                                                                                         \
        RCU_CUDA(dev, cudaFuncSetAttribute(KERN_, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(smem > 48 * 1024 ? smem : 48 * 1024))); \
        RCU_CUDA(dev, rcu_launch_cluster(dev, KERN_, grid, kThreads, smem, cluster ? n_splits : 0, a));                          \
    } while (0)
#define RCU_GS_C(NB_, EB_)                                              \
    do {                                                                \
        if (cluster) RCU_GS((grouped_step_mma_kernel<NB_, EB_, true>)); \
        else RCU_GS((grouped_step_mma_kernel<NB_, EB_, false>));        \
    } while (0)
    if (mma) {
        const int nb = a.D <= 64 ? 2 : a.D <= 128 ? 4 : 8;
        const size_t smem = (size_t)2 * kMmaHeads * (nb * 32 + 8) * 2 + (size_t)kWarps * nh * a.E * 4;
#define RCU_GS_E(NB_)                                                                     \
    do {                                                                                  \
        if (a.E <= 64) RCU_GS_C(NB_, 1);                                                  \
        else if (a.E <= 128) RCU_GS_C(NB_, 2);                                            \
        else RCU_GS_C(NB_, 4);                                                            \
    } while (0)
        if (nb == 2) RCU_GS_E(2);
        else if (nb == 4) RCU_GS_E(4);
        else RCU_GS_E(8);
#undef RCU_GS_E
    } else {
        const size_t smem = (size_t)kFmaHeads * a.D * 4 + (size_t)kTile * (a.D + a.E) * dt_esize(dt);
#define RCU_GS_T(T_)                                                     \
    do {                                                                 \
        if (a.E <= 64) RCU_GS((grouped_step_kernel<T_, 2>));             \
        else if (a.E <= 128) RCU_GS((grouped_step_kernel<T_, 4>));       \
        else if (a.E <= 256) RCU_GS((grouped_step_kernel<T_, 8>));       \
        else RCU_GS((grouped_step_kernel<T_, 16>));                      \
    } while (0)
        if (dt == RCU_F32) RCU_GS_T(float);
        else RCU_GS_T(__nv_bfloat16);
#undef RCU_GS_T
    }
#undef RCU_GS
#undef RCU_GS_C
    RCU_LAUNCH_CHECK(dev);
    return RCU_OK;
}

}  // namespace gstep
