// Fused decode step for a stack of parallel-residual layers whose mixers are linear attention with a state or latent
// attention with a sliding window, with stretches of layers that may be entered several times (each run of a layer has
// a state of its own).  The batch-1 counterpart of the lazy graph that runs prompts, over the same weights and states:
//
//   lightning run:  [norms + mixer projections + gated feed-forward inputs] -> [state update] -> [gated RMSNorm + both
//                   output projections + residual]
//   latent run:     [norms + low-rank projections + gated feed-forward inputs] -> [query expansion; latent append] ->
//                   [queries into latent space] -> [attention over latents] -> [merge + values] -> [both output
//                   projections + residual]
//
// Every matrix is streamed once by rows_kernel: a persistent grid of one CTA per SM; a team of 1, 2, 4 or 8 warps owns
// two rows at a time, keeps the next batch of 16-byte weight loads in flight while it multiplies the current one, and
// requests its first batch before it waits for the kernel before it (weights are constant, so programmatic dependent
// launch hides the start-up).  Norms, gates and activations are folded into the staging of the input vector in shared
// memory (f32) and into the row epilogues; activations stay in f32 between kernels.  Position and token live in device
// memory, so the whole step replays from one CUDA graph.
#include <algorithm>
#include <cmath>
#include <cstdlib>

#include "lm_math.cuh"

namespace {

constexpr int kThreads = 256, kWarps = 8;
constexpr int kRows = 2;            // rows per unit
constexpr int kBatch = 4;           // chunks of a row in flight per buffer
constexpr int kSub = 16;            // cached positions staged at a time
constexpr int kHeads = 8;           // heads per CTA of the latent attention (one warp each)
constexpr int kMaxSplits = 64;

enum { PRO_LAYER_NORM = 0, PRO_RMS, PRO_CONCAT, PRO_GATED_RMS };
enum { EPI_STORE = 0, EPI_MIXER_IN, EPI_RESIDUAL, EPI_BIAS };

struct RowsArgs {
    // weights: piece A rows [na, ka]; piece B: `pairs` gate rows followed by `pairs` up rows [2 pairs, kb] (not dual), or
    // rows [na, kb] multiplied by a second input and added to piece A's product (dual)
    const void *wa, *wb;
    int na, ka, pairs, kb, dual;
    int pro, epi;
    int split;                      // PRO_CONCAT: input A is x[0, split) followed by x2 (0: all of it is x, input B is x2)
    const float *x, *x2;            // input (x2: second input of PRO_CONCAT / PRO_GATED_RMS)
    const float *s1, *s2;           // norm scales
    const float* gate;              // PRO_GATED_RMS
    float eps, alpha;
    float *out, *out2;              // piece A rows; activated pairs
    const float *resid, *bias;
    int n_silu, n_sigmoid;          // EPI_MIXER_IN: rows below n_silu pass silu, rows from n_sigmoid on sigmoid
    int parts, aligned;
    // latent append, done by the first CTA (C == 0: none)
    const float* low;               // [C + R]
    const float *c_scale, *freqs;
    void* ring;
    int C, R, n_freq, ring_rows;
    float magnitude;
    const uint32_t* d_pos;
};

template <class T> __device__ __forceinline__ uint4 load_chunk(const T* row, int k, int K, bool aligned) {
    constexpr int VEC = 16 / (int)sizeof(T);
    if (k >= K) return make_uint4(0u, 0u, 0u, 0u);
    if (aligned) return ld_stream_v4(row + k);
    __align__(16) T v[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] = k + e < K ? row[k + e] : from_f32<T>(0.f);
    return *reinterpret_cast<const uint4*>(v);
}

// normalised latent and rotated key part of the current token into its ring row
template <class T> __device__ void append_latent(const RowsArgs& a, float* scratch) {
    float s = 0.f;
    for (int j = threadIdx.x; j < a.C; j += kThreads) s = fmaf(a.low[j], a.low[j], s);
    const float rstd = 1.0f / sqrtf(lm::block_sum(s, scratch) / (float)a.C + a.eps);
    const uint32_t p = *a.d_pos;
    T* row = reinterpret_cast<T*>(a.ring) + (size_t)(p % (uint32_t)a.ring_rows) * (a.C + a.R);
    for (int j = threadIdx.x; j < a.C; j += kThreads) row[j] = from_f32<T>(a.low[j] * rstd * a.c_scale[j]);
    const float* kr = a.low + a.C;
    for (int i = threadIdx.x; i < a.n_freq; i += kThreads) {
        const float2 cs = lm::rotary_angle(a.freqs, a.n_freq, i, p, a.magnitude);
        const float u = kr[2 * i], v = kr[2 * i + 1];
        row[a.C + 2 * i] = from_f32<T>(u * cs.x - v * cs.y);
        row[a.C + 2 * i + 1] = from_f32<T>(v * cs.x + u * cs.y);
    }
    for (int j = 2 * a.n_freq + threadIdx.x; j < a.R; j += kThreads) row[a.C + j] = from_f32<T>(kr[j]);
}

template <class T>
__global__ void __launch_bounds__(kThreads) rows_kernel(const RowsArgs a) {
    constexpr int VEC = 16 / (int)sizeof(T), CH = 32 * VEC;
    extern __shared__ __align__(16) float xs[];        // input A, padded to a multiple of 8; input B behind it
    __shared__ float scratch[32];
    __shared__ float red[kWarps][kRows];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int parts = a.parts, teams = kWarps / parts, team = warp / parts, part = warp % parts;
    const int ua = (a.na + kRows - 1) / kRows, units = ua + (a.dual ? 0 : a.pairs);
    const int xb = (a.ka + 7) & ~7;
    const int nca = (a.ka + CH - 1) / CH, ncb = (a.kb + CH - 1) / CH;
    const int gt = blockIdx.x * teams + team, gteams = gridDim.x * teams;

    // a unit's chunks: piece A's (or B's), in the dual form A's then B's; this warp takes chunks part, part + parts, ...
    auto chunks_of = [&](int u) { return a.dual ? nca + ncb : (u < ua ? nca : ncb); };
    auto row_ptr = [&](int u, int r, bool b_piece) -> const T* {
        if (a.dual || u < ua) {
            const int row = min(u * kRows + r, a.na - 1);
            return b_piece ? reinterpret_cast<const T*>(a.wb) + (size_t)row * a.kb : reinterpret_cast<const T*>(a.wa) + (size_t)row * a.ka;
        }
        return reinterpret_cast<const T*>(a.wb) + (size_t)(u - ua + r * a.pairs) * a.kb;
    };
    auto load_batch = [&](int u, int c0, uint4 (&w)[kBatch][kRows]) {
        const int nc = chunks_of(u);
#pragma unroll
        for (int i = 0; i < kBatch; ++i) {
            const int c = c0 + i * parts;
            const bool b_piece = a.dual ? c >= nca : u >= ua;
            const int k = (a.dual && b_piece ? c - nca : c) * CH + lane * VEC, K = b_piece ? a.kb : a.ka;
#pragma unroll
            for (int r = 0; r < kRows; ++r)
                w[i][r] = c < nc ? load_chunk<T>(row_ptr(u, r, b_piece), k, K, a.aligned) : make_uint4(0u, 0u, 0u, 0u);
        }
    };

    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    uint4 cur[kBatch][kRows];
    int u = gt, c0 = part;
    if (u < units) load_batch(u, c0, cur);
    asm volatile("griddepcontrol.wait;" ::: "memory");

    // ---- stage the input
    if (a.pro == PRO_LAYER_NORM || a.pro == PRO_RMS) {
        float s = 0.f;
        for (int j = threadIdx.x; j < a.ka; j += kThreads) {
            const float v = a.x[j];
            xs[j] = v;
            s += v;
        }
        const float mean = a.pro == PRO_LAYER_NORM ? lm::block_sum(s, scratch) / (float)a.ka : 0.f;
        float q = 0.f;
        for (int j = threadIdx.x; j < a.ka; j += kThreads) {
            const float d = xs[j] - mean;
            q = fmaf(d, d, q);
        }
        const float rstd = 1.0f / sqrtf(lm::block_sum(q, scratch) / (float)a.ka + a.eps);
        for (int j = threadIdx.x; j < a.ka; j += kThreads) {
            const float d = (xs[j] - mean) * rstd;
            xs[j] = d * a.s1[j];
            if (a.s2) xs[xb + j] = d * a.s2[j];
        }
    } else {
        float rstd = 1.f;
        if (a.pro == PRO_GATED_RMS) {
            float q = 0.f;
            for (int j = threadIdx.x; j < a.ka; j += kThreads) q = fmaf(a.x[j], a.x[j], q);
            rstd = 1.0f / sqrtf(lm::block_sum(q, scratch) / (float)a.ka + a.eps);
        }
        for (int j = threadIdx.x; j < a.ka; j += kThreads) {
            if (a.pro == PRO_GATED_RMS) xs[j] = a.x[j] * rstd * a.s1[j] * a.gate[j];
            else xs[j] = a.split && j >= a.split ? a.x2[j - a.split] : a.x[j];
        }
        for (int j = threadIdx.x; j < a.kb; j += kThreads) xs[xb + j] = a.x2[j];
    }
    for (int j = a.ka + threadIdx.x; j < xb; j += kThreads) xs[j] = 0.f;
    for (int j = a.kb + threadIdx.x; j < ((a.kb + 7) & ~7); j += kThreads) xs[xb + j] = 0.f;
    if (a.C > 0 && blockIdx.x == 0) append_latent<T>(a, scratch);
    __syncthreads();

    // ---- rows
    float acc[kRows] = {};
    while (u < units) {
        const int nc = chunks_of(u);
        int nu = u, n0 = c0 + kBatch * parts;
        const bool last = n0 >= nc;
        if (last) { nu = u + gteams; n0 = part; }
        uint4 next[kBatch][kRows];
        if (nu < units) load_batch(nu, n0, next);
#pragma unroll
        for (int i = 0; i < kBatch; ++i) {
            const int c = c0 + i * parts;
            if (c >= nc) break;
            const bool b_piece = a.dual ? c >= nca : u >= ua;
            const int k = (a.dual && b_piece ? c - nca : c) * CH + lane * VEC;
            if (k < (b_piece ? a.kb : a.ka)) {
                const float* xv = xs + (b_piece ? xb : 0) + k;
                float f[VEC];
#pragma unroll
                for (int e = 0; e < VEC; e += 4) *reinterpret_cast<float4*>(f + e) = *reinterpret_cast<const float4*>(xv + e);
#pragma unroll
                for (int r = 0; r < kRows; ++r) {
                    const T* wv = reinterpret_cast<const T*>(&cur[i][r]);
#pragma unroll
                    for (int e = 0; e < VEC; ++e) acc[r] = fmaf(to_f32<T>(wv[e]), f[e], acc[r]);
                }
            }
        }
        if (last) {
#pragma unroll
            for (int r = 0; r < kRows; ++r) acc[r] = warp_sum(acc[r]);
            if (parts > 1) {
                if (lane == 0) {
#pragma unroll
                    for (int r = 0; r < kRows; ++r) red[warp][r] = acc[r];
                }
                asm volatile("bar.sync %0, %1;" ::"r"(1 + team), "r"(parts * 32) : "memory");
                if (part == 0) {
#pragma unroll
                    for (int r = 0; r < kRows; ++r) {
                        acc[r] = 0.f;
                        for (int q = 0; q < parts; ++q) acc[r] += red[team * parts + q][r];
                    }
                }
                asm volatile("bar.sync %0, %1;" ::"r"(1 + team), "r"(parts * 32) : "memory");
            }
            if (part == 0 && lane == 0) {
                if (a.dual || u < ua) {
#pragma unroll
                    for (int r = 0; r < kRows; ++r) {
                        const int row = u * kRows + r;
                        if (row >= a.na) break;
                        float v = acc[r];
                        if (a.epi == EPI_MIXER_IN) {
                            if (row < a.n_silu) v = lm::silu(v);
                            else if (row >= a.n_sigmoid) v = lm::sigmoid(v);
                        } else if (a.epi == EPI_RESIDUAL) {
                            v = fmaf(a.alpha, v, a.resid[row]);
                        } else if (a.epi == EPI_BIAS) {
                            v += a.bias[row];
                        }
                        a.out[row] = v;
                    }
                } else {
                    a.out2[u - ua] = lm::gelu_tanh(acc[0]) * acc[1];
                }
            }
#pragma unroll
            for (int r = 0; r < kRows; ++r) acc[r] = 0.f;
        }
        u = nu;
        c0 = n0;
#pragma unroll
        for (int i = 0; i < kBatch; ++i)
#pragma unroll
            for (int r = 0; r < kRows; ++r) cur[i][r] = next[i][r];
    }
}

// x0 = x = embedding row of the token; an id outside the table is clamped and flagged
template <class T>
__global__ void __launch_bounds__(kThreads) embed_kernel(const int32_t* token, const T* __restrict__ table, int vocab, int width, float* x0, float* x,
                                                         int* status) {
    rcu_kernel_entry();
    int t = *token;
    if (t < 0 || t >= vocab) {
        if (threadIdx.x == 0 && blockIdx.x == 0) atomicOr(status, RCU_DEVFLAG_BOUNDS);
        t = t < 0 ? 0 : vocab - 1;
    }
    for (int j = blockIdx.x * kThreads + threadIdx.x; j < width; j += gridDim.x * kThreads) {
        const float v = to_f32<T>(table[(size_t)t * width + j]);
        x0[j] = v;
        x[j] = v;
    }
}

// One token of linear attention: CTA = (head, 32 value columns), lane = column, warp = every eighth feature row.
__global__ void __launch_bounds__(kThreads) lightning_step_kernel(const float* __restrict__ mix, const float* __restrict__ decay, float* __restrict__ state,
                                                                  float* __restrict__ out, int H, int D, int E) {
    rcu_kernel_entry();
    __shared__ float part[kWarps][32];
    const int h = blockIdx.x, lane = threadIdx.x & 31, g = threadIdx.x >> 5;
    const int e = blockIdx.y * 32 + lane;
    const float* q = mix + (size_t)h * D;
    const float* k = q + (size_t)H * D;
    const float v = e < E ? mix[(size_t)2 * H * D + (size_t)h * E + e] : 0.f;
    const float dec = decay[h];
    float* S = state + (size_t)h * D * E;
    float o = 0.f;
    if (e < E) {
#pragma unroll 4
        for (int d = g; d < D; d += kWarps) {
            const float s = fmaf(dec, S[(size_t)d * E + e], k[d] * v);
            S[(size_t)d * E + e] = s;
            o = fmaf(q[d], s, o);
        }
    }
    part[g][lane] = o;
    __syncthreads();
    if (g == 0 && e < E) {
        o = 0.f;
#pragma unroll
        for (int w = 0; w < kWarps; ++w) o += part[w][lane];
        out[(size_t)h * E + e] = o;
    }
}

// Queries into latent space: qa[h] = scale * [W_uk[h]^T q_h, rotate(q_h's rotated part)].  CTA = (head, 32 latent columns).
template <class T>
__global__ void __launch_bounds__(kThreads) absorb_kernel(const float* __restrict__ q, const T* __restrict__ uk, const float* __restrict__ freqs, int n_freq,
                                                          float magnitude, const uint32_t* d_pos, float* __restrict__ qa, int D, int R, int C, float scale) {
    rcu_kernel_entry();
    __shared__ float part[kWarps][32];
    const int h = blockIdx.x, lane = threadIdx.x & 31, g = threadIdx.x >> 5;
    const int c = blockIdx.y * 32 + lane;
    const float* qh = q + (size_t)h * (D + R);
    float* dst = qa + (size_t)h * (C + R);
    float acc = 0.f;
    if (c < C) {
        const T* w = uk + (size_t)h * D * C + c;
#pragma unroll 8
        for (int d = g; d < D; d += kWarps) acc = fmaf(to_f32<T>(w[(size_t)d * C]), qh[d], acc);
    }
    part[g][lane] = acc;
    __syncthreads();
    if (g == 0 && c < C) {
        acc = 0.f;
#pragma unroll
        for (int w = 0; w < kWarps; ++w) acc += part[w][lane];
        dst[c] = acc * scale;
    }
    if (blockIdx.y == 0) {
        const uint32_t p = *d_pos;
        for (int i = threadIdx.x; i < n_freq; i += kThreads) {
            const float2 cs = lm::rotary_angle(freqs, n_freq, i, p, magnitude);
            const float u = qh[D + 2 * i], v = qh[D + 2 * i + 1];
            dst[C + 2 * i] = (u * cs.x - v * cs.y) * scale;
            dst[C + 2 * i + 1] = (v * cs.x + u * cs.y) * scale;
        }
        for (int j = 2 * n_freq + threadIdx.x; j < R; j += kThreads) dst[C + j] = qh[D + j] * scale;
    }
}

// Attention of one token over the cached latents: CTA = (run of positions, eight heads), a warp per head.  Positions are
// staged kSub at a time in shared memory and shared by the heads; each warp keeps an online softmax and its share of the
// weighted latents.  partial[split][head]: C sums, then the maximum and the sum of the weights.
template <class T, int PC>
__global__ void __launch_bounds__(kThreads) latent_step_kernel(const float* __restrict__ qa, const T* __restrict__ ring, int ring_rows, int window,
                                                               const uint32_t* d_pos, float* __restrict__ partial, int H, int C, int R) {
    rcu_kernel_entry();
    extern __shared__ __align__(16) float q_s[];         // [kHeads][C + R], then the staged rows
    const int W = C + R, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    T* rows = reinterpret_cast<T*>(q_s + (size_t)kHeads * W);
    const int h0 = blockIdx.y * kHeads, h = h0 + warp;
    const int pos = (int)*d_pos, first = max(0, pos - window + 1), n = pos - first + 1;
    const int per = (n + gridDim.x - 1) / gridDim.x;
    const int begin = first + min(n, (int)blockIdx.x * per), end = first + min(n, ((int)blockIdx.x + 1) * per);
    for (int j = threadIdx.x; j < min(kHeads, H - h0) * W; j += kThreads) q_s[j] = qa[(size_t)h0 * W + j];
    const float* q = q_s + (size_t)warp * W;
    float m = -INFINITY, l = 0.f, o[PC];
#pragma unroll
    for (int c = 0; c < PC; ++c) o[c] = 0.f;
    for (int p0 = begin; p0 < end; p0 += kSub) {
        const int np = min(kSub, end - p0);
        __syncthreads();
        for (int j = threadIdx.x; j < np * W; j += kThreads) {
            const int r = j / W;
            rows[j] = ring[(size_t)((p0 + r) % ring_rows) * W + (j - r * W)];
        }
        __syncthreads();
        if (h >= H) continue;
        float s[kSub];
#pragma unroll
        for (int r = 0; r < kSub; ++r) s[r] = 0.f;
        for (int c = lane; c < W; c += 32) {
            const float qv = q[c];
#pragma unroll
            for (int r = 0; r < kSub; ++r)
                if (r < np) s[r] = fmaf(qv, to_f32<T>(rows[r * W + c]), s[r]);
        }
        float mt = -INFINITY;
#pragma unroll
        for (int r = 0; r < kSub; ++r) {
            s[r] = r < np ? warp_sum(s[r]) : -INFINITY;
            mt = fmaxf(mt, s[r]);
        }
        const float mn = fmaxf(m, mt), corr = expf(m - mn);
        l *= corr;
#pragma unroll
        for (int c = 0; c < PC; ++c) o[c] *= corr;
#pragma unroll
        for (int r = 0; r < kSub; ++r) {
            s[r] = expf(s[r] - mn);
            l += s[r];
        }
        m = mn;
#pragma unroll
        for (int r = 0; r < kSub; ++r) {
            if (r >= np) break;
#pragma unroll
            for (int c = 0; c < PC; ++c)
                if (lane + 32 * c < C) o[c] = fmaf(s[r], to_f32<T>(rows[r * W + lane + 32 * c]), o[c]);
        }
    }
    if (h >= H) return;
    float* dst = partial + ((size_t)blockIdx.x * H + h) * (C + 2);
#pragma unroll
    for (int c = 0; c < PC; ++c)
        if (lane + 32 * c < C) dst[lane + 32 * c] = o[c];
    if (lane == 0) {
        dst[C] = m;
        dst[C + 1] = l;
    }
}

// Merge of a head's partial results and its values: out[h] = W_uv[h] . (weighted latent).  CTA = (head, run of value rows).
template <class T>
__global__ void __launch_bounds__(kThreads) latent_values_kernel(const float* __restrict__ partial, int splits, const T* __restrict__ uv, float* __restrict__ out,
                                                                 int H, int C, int E, int rows_per) {
    rcu_kernel_entry();
    extern __shared__ float c_s[];
    __shared__ float wgt[kMaxSplits];
    const int h = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const float* ph = partial + (size_t)h * (C + 2);
    const size_t stride = (size_t)H * (C + 2);
    if (warp == 0) {
        float m0 = lane < splits ? ph[lane * stride + C] : -INFINITY, m1 = lane + 32 < splits ? ph[(lane + 32) * stride + C] : -INFINITY;
        const float M = warp_max(fmaxf(m0, m1));
        const float w0 = lane < splits ? expf(m0 - M) : 0.f, w1 = lane + 32 < splits ? expf(m1 - M) : 0.f;
        float l = (lane < splits ? w0 * ph[lane * stride + C + 1] : 0.f) + (lane + 32 < splits ? w1 * ph[(lane + 32) * stride + C + 1] : 0.f);
        l = warp_sum(l);
        wgt[lane] = w0 / l;
        wgt[lane + 32] = w1 / l;
    }
    __syncthreads();
    for (int c = threadIdx.x; c < C; c += kThreads) {
        float s = 0.f;
#pragma unroll 8
        for (int i = 0; i < splits; ++i) s = fmaf(wgt[i], ph[i * stride + c], s);
        c_s[c] = s;
    }
    __syncthreads();
    const int e1 = min(E, ((int)blockIdx.y + 1) * rows_per);
    for (int e = blockIdx.y * rows_per + warp; e < e1; e += kWarps) {
        const T* w = uv + ((size_t)h * E + e) * C;
        float acc = 0.f;
#pragma unroll 4
        for (int c = lane; c < C; c += 32) acc = fmaf(to_f32<T>(w[c]), c_s[c], acc);
        acc = warp_sum(acc);
        if (lane == 0) out[(size_t)h * E + e] = acc;
    }
}

// arg-max (the first maximum wins) and the step to the next position
__global__ void __launch_bounds__(1024) argmax_next_kernel(const float* __restrict__ logits, int n, int32_t* out, uint32_t* d_pos) {
    rcu_kernel_entry();
    __shared__ float bv[32];
    __shared__ int bi[32];
    if (out) {
        float best = -INFINITY;
        int idx = 0x7fffffff;
        for (int i = threadIdx.x; i < n; i += 1024)
            if (logits[i] > best || idx == 0x7fffffff) { best = logits[i]; idx = i; }
#pragma unroll
        for (int pass = 0; pass < 2; ++pass) {
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) {
                const float ov = __shfl_xor_sync(0xffffffffu, best, o);
                const int oi = __shfl_xor_sync(0xffffffffu, idx, o);
                if (ov > best || (ov == best && oi < idx)) { best = ov; idx = oi; }
            }
            if (pass == 0) {
                if ((threadIdx.x & 31) == 0) { bv[threadIdx.x >> 5] = best; bi[threadIdx.x >> 5] = idx; }
                __syncthreads();
                best = bv[threadIdx.x & 31];
                idx = bi[threadIdx.x & 31];
            }
        }
        if (threadIdx.x == 0) *out = min(idx, n - 1);
    }
    if (threadIdx.x == 0) *d_pos += 1;
}

__global__ void set_position_kernel(uint32_t* p, uint32_t v) {
    rcu_kernel_entry();
    *p = v;
}

}  // namespace

struct rcu_stack {
    rcu_device* dev;
    rcu_stack_config cfg;
    std::vector<rcu_stack_run> runs;
    const void *embed, *head;
    const float* final_norm;
    float* pool = nullptr;              // every f32 vector below
    float *x0, *xa, *xb, *mix, *act, *y, *q, *qa, *partial, *logits;
    uint32_t* d_pos = nullptr;
    uint32_t position = 0, kernels_per_step = 0;
    uint64_t steps = 0;
    cudaGraphExec_t graph_exec = nullptr;
    const int32_t* cap_token = nullptr;
    void* cap_logits = nullptr;
    int32_t* cap_argmax = nullptr;
};

namespace {

int latent_splits(const rcu_stack_run& r) { return (int)std::min<uint32_t>(kMaxSplits, std::max<uint32_t>(1, (std::min(r.window, r.ring_rows) + kSub - 1) / kSub)); }

// warps per team: fewest warp steps over the whole grid
int plan_parts(int grid, int units, int nc) {
    int best = 1;
    long long best_cost = -1;
    for (int parts = 1; parts <= kWarps; parts *= 2) {
        const long long teams = (long long)grid * (kWarps / parts), rounds = (units + teams - 1) / teams;
        const long long cost = rounds * ((((nc + parts - 1) / parts) + kBatch - 1) / kBatch * kBatch);
        if (best_cost < 0 || cost < best_cost) { best = parts; best_cost = cost; }
    }
    return best;
}

template <class T> rcu_status launch_rows(rcu_device* dev, RowsArgs a) {
    constexpr int VEC = 16 / (int)sizeof(T), CH = 32 * VEC;
    const int units = (a.na + kRows - 1) / kRows + (a.dual ? 0 : a.pairs);
    const int nca = (a.ka + CH - 1) / CH, ncb = (a.kb + CH - 1) / CH;
    a.parts = plan_parts(dev->sm_count, units, a.dual ? nca + ncb : std::max(nca, ncb));
    const bool has_b = a.kb > 0 && a.wb;
    a.aligned = a.ka % VEC == 0 && (!has_b || a.kb % VEC == 0) && ((reinterpret_cast<uintptr_t>(a.wa) | reinterpret_cast<uintptr_t>(a.wb)) & 15) == 0;
    const int teams = kWarps / a.parts;
    const int grid = std::max(1, std::min(dev->sm_count, (units + teams - 1) / teams));
    const size_t smem = ((size_t)((a.ka + 7) & ~7) + (size_t)((a.kb + 7) & ~7)) * 4;
    if (smem + 1024 > (size_t)dev->smem_optin) return rcu_fail(dev, RCU_ERR_UNSUPPORTED, "stack: input vectors of %d + %d do not fit shared memory", a.ka, a.kb);
    RCU_CUDA(dev, cudaFuncSetAttribute(rows_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)std::max(smem, (size_t)(64 * 1024))));
    RCU_CUDA(dev, rcu_launch(dev, rows_kernel<T>, grid, kThreads, smem, a));
    RCU_LAUNCH_CHECK(dev);
    return RCU_OK;
}

template <class T> rcu_status launch_latent_step(rcu_device* dev, const rcu_stack* s, const rcu_stack_run& r) {
    const int H = (int)r.heads, C = (int)r.kv_rank, R = (int)r.rot_dim, splits = latent_splits(r);
    const size_t smem = (size_t)kHeads * (C + R) * 4 + (size_t)kSub * (C + R) * sizeof(T);
    const dim3 grid(splits, (H + kHeads - 1) / kHeads);
#define RCU_LS(PC_)                                                                                                                              \
    do {                                                                                                                                         \
        RCU_CUDA(dev, cudaFuncSetAttribute(latent_step_kernel<T, PC_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)std::max(smem, (size_t)(48 * 1024)))); \
        RCU_CUDA(dev, rcu_launch(dev, latent_step_kernel<T, PC_>, grid, kThreads, smem, s->qa, (const T*)r.state, (int)r.ring_rows, (int)r.window, s->d_pos, \
                                 s->partial, H, C, R));                                                                                          \
    } while (0)
    if (C <= 128) RCU_LS(4);
    else if (C <= 256) RCU_LS(8);
    else if (C <= 512) RCU_LS(16);
    else RCU_LS(32);
#undef RCU_LS
    RCU_LAUNCH_CHECK(dev);
    return RCU_OK;
}

#define STACK_TRY(expr)                          \
    do {                                         \
        const rcu_status st_ = (expr);           \
        if (st_ != RCU_OK) return st_;           \
    } while (0)

template <class T> rcu_status run_step(rcu_stack* s, const int32_t* token, float* logits, int32_t* argmax) {
    rcu_device* dev = s->dev;
    const rcu_stack_config& c = s->cfg;
    const int W = (int)c.width;
    float *x = s->xa, *other = s->xb;
    RCU_CUDA(dev, rcu_launch(dev, embed_kernel<T>, (W + kThreads - 1) / kThreads, kThreads, 0, token, (const T*)s->embed, (int)c.vocab, W, s->x0, x, dev->d_status));
    RCU_LAUNCH_CHECK(dev);
    for (const rcu_stack_run& r : s->runs) {
        if (r.enter) {                          // x <- W_enter [x; x0] + step
            RowsArgs a = {};
            a.wa = r.enter; a.na = W; a.ka = 2 * W;
            a.pro = PRO_CONCAT; a.epi = EPI_BIAS;
            a.x = x; a.x2 = s->x0; a.split = W;
            a.bias = (const float*)r.enter_bias; a.out = other;
            STACK_TRY(launch_rows<T>(dev, a));
            std::swap(x, other);
        }
        const int H = (int)r.heads, D = (int)r.dim, E = (int)r.vdim, ff = (int)r.ff;
        RowsArgs in = {};
        in.wa = r.mix_in; in.ka = W; in.wb = r.gate_up; in.pairs = ff; in.kb = ff ? W : 0;
        in.pro = PRO_LAYER_NORM; in.x = x; in.s1 = (const float*)r.norm1; in.s2 = ff ? (const float*)r.norm2 : nullptr; in.eps = c.eps;
        in.out = s->mix; in.out2 = s->act;
        RowsArgs out = {};
        out.wa = r.out; out.na = W; out.ka = H * E; out.wb = r.down; out.kb = ff; out.dual = 1;
        out.x2 = s->act; out.eps = c.eps; out.epi = EPI_RESIDUAL; out.alpha = c.residual_mult; out.resid = x; out.out = x;
        if (r.mixer == RCU_MIXER_LIGHTNING) {
            in.na = 2 * H * D + 2 * H * E;
            in.epi = EPI_MIXER_IN; in.n_silu = 2 * H * D + H * E; in.n_sigmoid = in.n_silu;
            STACK_TRY(launch_rows<T>(dev, in));
            RCU_CUDA(dev, rcu_launch(dev, lightning_step_kernel, dim3(H, (E + 31) / 32), kThreads, 0, s->mix, (const float*)r.decay, (float*)r.state, s->y, H, D, E));
            RCU_LAUNCH_CHECK(dev);
            out.pro = PRO_GATED_RMS; out.x = s->y; out.s1 = (const float*)r.mix_norm; out.gate = s->mix + 2 * H * D + H * E;
        } else {
            const int Q = (int)r.q_rank, C = (int)r.kv_rank, R = (int)r.rot_dim, nf = (int)r.rot_pairs;
            in.na = Q + C + R;
            in.epi = EPI_STORE;
            STACK_TRY(launch_rows<T>(dev, in));
            RowsArgs uq = {};
            uq.wa = r.uq; uq.na = H * (D + R); uq.ka = Q; uq.pro = PRO_RMS; uq.x = s->mix; uq.s1 = (const float*)r.mix_norm; uq.eps = c.eps; uq.out = s->q;
            uq.low = s->mix + Q; uq.c_scale = (const float*)r.kv_norm; uq.freqs = (const float*)r.freqs; uq.ring = r.state; uq.C = C; uq.R = R; uq.n_freq = nf;
            uq.ring_rows = (int)r.ring_rows; uq.magnitude = r.rot_magnitude; uq.d_pos = s->d_pos;
            STACK_TRY(launch_rows<T>(dev, uq));
            RCU_CUDA(dev, rcu_launch(dev, absorb_kernel<T>, dim3(H, (C + 31) / 32), kThreads, 0, s->q, (const T*)r.ukv, (const float*)r.freqs, nf, r.rot_magnitude,
                                     s->d_pos, s->qa, D, R, C, r.scale));
            RCU_LAUNCH_CHECK(dev);
            STACK_TRY(launch_latent_step<T>(dev, s, r));
            const int per = 16;
            RCU_CUDA(dev, rcu_launch(dev, latent_values_kernel<T>, dim3(H, (E + per - 1) / per), kThreads, (size_t)C * 4, s->partial, latent_splits(r),
                                     (const T*)r.ukv + (size_t)H * D * C, s->y, H, C, E, per));
            RCU_LAUNCH_CHECK(dev);
            out.pro = PRO_CONCAT; out.x = s->y;
        }
        STACK_TRY(launch_rows<T>(dev, out));
    }
    RowsArgs head = {};
    head.wa = s->head; head.na = (int)c.vocab; head.ka = W; head.pro = PRO_LAYER_NORM; head.x = x; head.s1 = s->final_norm; head.eps = c.eps; head.out = logits;
    STACK_TRY(launch_rows<T>(dev, head));
    RCU_CUDA(dev, rcu_launch(dev, argmax_next_kernel, 1, 1024, 0, logits, (int)c.vocab, argmax, s->d_pos));
    RCU_LAUNCH_CHECK(dev);
    return RCU_OK;
}

rcu_status run_any(rcu_stack* s, const int32_t* token, float* logits, int32_t* argmax) {
    return s->cfg.weight_dt == RCU_F32 ? run_step<float>(s, token, logits, argmax) : run_step<__nv_bfloat16>(s, token, logits, argmax);
}

}  // namespace

extern "C" {

rcu_status rcu_stack_create(rcu_device* dev, const rcu_stack_config* cfg, const rcu_stack_run* runs, const void* embed, const void* final_norm,
                            const void* head, rcu_stack** out) {
    if (!dev || !cfg || !runs || !embed || !final_norm || !head || !out) return RCU_ERR_INVALID_ARG;
    RCU_REQUIRE(dev, cfg->weight_dt == RCU_BF16 || cfg->weight_dt == RCU_F32, "stack: weights are bf16 or f32");
    RCU_REQUIRE(dev, cfg->width > 0 && cfg->vocab > 0 && cfg->n_runs > 0, "stack: empty model");
    size_t mix = 0, act = 1, y = 0, q = 1, qa = 1, partial = 1;
    for (uint32_t i = 0; i < cfg->n_runs; ++i) {
        const rcu_stack_run& r = runs[i];
        RCU_REQUIRE(dev, r.norm1 && r.mix_in && r.mix_norm && r.out && r.state && r.heads && r.dim && r.vdim, "stack: run %u lacks a weight or a size", i);
        RCU_REQUIRE(dev, r.ff == 0 || (r.norm2 && r.gate_up && r.down), "stack: run %u lacks a feed-forward weight", i);
        RCU_REQUIRE(dev, r.heads <= 65535, "stack: run %u has too many heads", i);
        if (r.mixer == RCU_MIXER_LIGHTNING) {
            RCU_REQUIRE(dev, r.decay, "stack: run %u has no decay", i);
            mix = std::max(mix, (size_t)r.heads * 2 * (r.dim + r.vdim));
        } else {
            RCU_REQUIRE(dev, r.mixer == RCU_MIXER_LATENT, "stack: run %u has an unknown mixer", i);
            RCU_REQUIRE(dev, r.q_rank && r.kv_rank && r.kv_norm && r.uq && r.ukv && (r.rot_pairs == 0 || r.freqs) && 2 * r.rot_pairs <= r.rot_dim,
                        "stack: run %u lacks a weight or a size", i);
            RCU_REQUIRE(dev, r.window > 0 && r.ring_rows > 0, "stack: run %u has no window", i);
            if (r.kv_rank > 1024) return rcu_fail(dev, RCU_ERR_UNSUPPORTED, "stack: latents of %u (at most 1024)", r.kv_rank);
            mix = std::max(mix, (size_t)r.q_rank + r.kv_rank + r.rot_dim);
            q = std::max(q, (size_t)r.heads * (r.dim + r.rot_dim));
            qa = std::max(qa, (size_t)r.heads * (r.kv_rank + r.rot_dim));
            partial = std::max(partial, (size_t)latent_splits(r) * r.heads * (r.kv_rank + 2));
        }
        act = std::max(act, (size_t)r.ff);
        y = std::max(y, (size_t)r.heads * r.vdim);
    }
    DevGuard g(dev->ordinal);
    rcu_stack* s = new rcu_stack();
    s->dev = dev;
    s->cfg = *cfg;
    s->runs.assign(runs, runs + cfg->n_runs);
    s->embed = embed; s->head = head; s->final_norm = (const float*)final_norm;
    const size_t sizes[] = {cfg->width, cfg->width, cfg->width, mix, act, y, q, qa, partial};
    float** ptrs[] = {&s->x0, &s->xa, &s->xb, &s->mix, &s->act, &s->y, &s->q, &s->qa, &s->partial};
    size_t total = 64;
    for (size_t n : sizes) total += (n + 63) & ~(size_t)63;
    void* p = nullptr;
    rcu_status st = rcu_alloc(dev, total * 4, &p);
    if (st != RCU_OK) { delete s; return st; }
    s->pool = (float*)p;
    s->d_pos = (uint32_t*)p;
    float* at = s->pool + 64;
    for (size_t i = 0; i < sizeof(sizes) / sizeof(sizes[0]); ++i) {
        *ptrs[i] = at;
        at += (sizes[i] + 63) & ~(size_t)63;
    }
    st = rcu_stack_set_position(s, 0);
    if (st != RCU_OK) { rcu_free(dev, p); delete s; return st; }
    *out = s;
    return RCU_OK;
}

void rcu_stack_destroy(rcu_stack* s) {
    if (!s) return;
    DevGuard g(s->dev->ordinal);
    cudaStreamSynchronize(s->dev->stream);
    if (s->graph_exec) cudaGraphExecDestroy(s->graph_exec);
    rcu_free(s->dev, s->pool);
    delete s;
}

rcu_status rcu_stack_set_position(rcu_stack* s, uint32_t position) {
    if (!s) return RCU_ERR_INVALID_ARG;
    DevGuard g(s->dev->ordinal);
    rcu_launch(s->dev, set_position_kernel, 1, 1, 0, s->d_pos, position);
    RCU_LAUNCH_CHECK(s->dev);
    s->position = position;
    return RCU_OK;
}

uint32_t rcu_stack_position(const rcu_stack* s) { return s ? s->position : 0; }
uint32_t rcu_stack_kernels_per_step(const rcu_stack* s) { return s ? s->kernels_per_step : 0; }

rcu_status rcu_stack_step(rcu_stack* s, const int32_t* token_dev, float* logits_dev, int32_t* argmax_dev) {
    if (!s || !token_dev || !logits_dev) return RCU_ERR_INVALID_ARG;
    rcu_device* dev = s->dev;
    for (const rcu_stack_run& r : s->runs)
        RCU_REQUIRE(dev, r.mixer != RCU_MIXER_LATENT || r.ring_rows >= r.window || s->position < r.ring_rows, "stack: the latent cache is full (%u rows)", r.ring_rows);
    DevGuard g(dev->ordinal);
    const bool use_graph = std::getenv("RCU_NO_GRAPH") == nullptr && dev->stream != nullptr;
    if (!use_graph || s->steps == 0) {      // the first step sets kernel attributes and counts the launches
        const uint64_t l0 = dev->launches;
        STACK_TRY(run_any(s, token_dev, logits_dev, argmax_dev));
        s->kernels_per_step = (uint32_t)(dev->launches - l0);
    } else {
        if (!s->graph_exec || s->cap_token != token_dev || s->cap_logits != logits_dev || s->cap_argmax != argmax_dev) {
            if (s->graph_exec) { cudaGraphExecDestroy(s->graph_exec); s->graph_exec = nullptr; }
            cudaGraph_t graph = nullptr;
            const uint64_t l0 = dev->launches;
            RCU_CUDA(dev, cudaStreamBeginCapture(dev->stream, cudaStreamCaptureModeThreadLocal));
            const rcu_status st = run_any(s, token_dev, logits_dev, argmax_dev);
            cudaError_t e = cudaStreamEndCapture(dev->stream, &graph);
            dev->launches = l0;             // capture launched nothing
            if (st != RCU_OK) { if (graph) cudaGraphDestroy(graph); return st; }
            if (e != cudaSuccess) return rcu_fail(dev, RCU_ERR_CUDA, "stack: graph capture failed: %s", cudaGetErrorString(e));
            e = cudaGraphInstantiate(&s->graph_exec, graph, 0);
            cudaGraphDestroy(graph);
            if (e != cudaSuccess) return rcu_fail(dev, RCU_ERR_CUDA, "stack: graph instantiation failed: %s", cudaGetErrorString(e));
            s->cap_token = token_dev; s->cap_logits = logits_dev; s->cap_argmax = argmax_dev;
        }
        RCU_CUDA(dev, cudaGraphLaunch(s->graph_exec, dev->stream));
        dev->launches += s->kernels_per_step;
    }
    s->steps++;
    s->position++;
    return RCU_OK;
}

}  // extern "C"
