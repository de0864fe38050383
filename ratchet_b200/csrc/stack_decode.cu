// Fused decode step for a stack of layers whose mixers are linear attention with a state, latent attention with a sliding
// window or attention of grouped heads, with stretches of layers that may be entered several times (each run of a layer has
// a state of its own).  The batch-1 counterpart of the lazy graph that runs prompts, over the same weights and states.
// Parallel-residual layers (norm before the sublayers, which share their input and are added together):
//
//   lightning run:  [norms + mixer projections + gated feed-forward inputs] -> [state update] -> [gated RMSNorm + both
//                   output projections + residual]
//   latent run:     [norms + low-rank projections + gated feed-forward inputs] -> [query expansion; latent append] ->
//                   [queries into latent space] -> [attention over latents] -> [merge + values] -> [both output
//                   projections + residual]
//
// Layers with a norm on each sublayer's output (grouped_step.cuh has the attention kernels):
//
//   grouped run:    [q, k, v rows] -> [head norms, rotation, append, attention, merge] -> [output rows] -> [up rows, squared relu] ->
//                   [down rows], where the first and fourth begin by adding the normed output of the sublayer before to the
//                   residual stream - every CTA for itself, the first one stores the sum for those that follow.
//
// Every matrix is streamed once.  bf16 weights whose rows are whole 64-element blocks take rows_mma_kernel: a persistent
// grid of one CTA per SM, sixteen rows per unit, a team of 1, 2, 4 or 8 warps sharing a unit's columns.  Each warp keeps a ring
// of shared-memory slots filled by TMA (16 rows x 128 columns, 128-byte swizzle, mbarrier transaction counts) and fills it
// before it waits for the kernel before it: weights are constant, so with programmatic dependent launch the first rows
// travel as soon as that kernel leaves an SM.  The products run on the tensor cores as 16 x 16 times 16 x 8 with the input vector as
// two of the eight columns - its bf16 rounding and the remainder, so that activations keep 16 bits of mantissa - because
// unpacking bf16 weights for FFMA costs more issue slots than the memory system leaves.  f32 weights and other row lengths
// take rows_kernel (FFMA, plain loads).  Norms, gates and activations are folded into the staging of the input vector in
// shared memory and into the row epilogues; activations stay in f32 between kernels.  Position and token live in device
// memory, so the whole step replays from one CUDA graph.
#include <algorithm>
#include <cmath>
#include <cstdlib>

#include "bulk_async.cuh"
#include "grouped_step.cuh"
#include "lm_mma.cuh"

namespace {

constexpr int kThreads = 256, kWarps = 8;
constexpr int kRows = 2;            // rows per unit of rows_kernel
constexpr int kUnit = 16;           // rows per unit of rows_mma_kernel
constexpr int kItem = 128;          // columns per ring slot
constexpr int kSlotBytes = kUnit * kItem * 2;
constexpr int kMaxSlots = 8;
constexpr int kSub = 16;            // cached positions staged at a time
constexpr int kHeads = 8;           // heads per CTA of the latent attention (one warp each)
constexpr int kMaxSplits = 64;

enum { PRO_LAYER_NORM = 0, PRO_RMS, PRO_CONCAT, PRO_GATED_RMS, PRO_POST_NORM };
enum { EPI_STORE = 0, EPI_MIXER_IN, EPI_RESIDUAL, EPI_BIAS, EPI_RELU_SQUARED, EPI_SOFTCAP };

struct RowsArgs {
    // weights: piece A rows [na, ka]; piece B: `pairs` gate rows followed by `pairs` up rows [2 pairs, kb] (not dual), or
    // rows [na, kb] multiplied by a second input and added to piece A's product (dual)
    const void *wa, *wb;
    int na, ka, pairs, kb, dual;
    int pro, epi;
    int split;                      // PRO_CONCAT: input A is x[0, split) followed by x2 (0: all of it is x, input B is x2)
    const float *x, *x2;            // input (x2: second input of PRO_CONCAT / PRO_GATED_RMS; sublayer output of PRO_POST_NORM)
    const float *s1, *s2;           // norm scales (PRO_POST_NORM: of the sublayer norm, of a LayerNorm of the sum or null)
    const float *b1, *b2;           // their shifts (nullable)
    float* x_out;                   // PRO_POST_NORM: the first CTA stores the sum here (nullable)
    const float* gate;              // PRO_GATED_RMS
    float eps, alpha;
    float *out, *out2;              // piece A rows; activated pairs
    const float *resid, *bias;
    int n_silu, n_sigmoid;          // EPI_MIXER_IN: rows below n_silu pass silu, rows from n_sigmoid on sigmoid
    int parts, slots;               // warps per team; ring slots per warp
    int* status;
    // latent append, done by the first CTA (C == 0: none)
    const float* low;               // [C + R]
    const float *c_scale, *freqs;
    void* ring;
    int C, R, n_freq, ring_rows;
    float magnitude;
    const uint32_t* d_pos;
};

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

__host__ __device__ __forceinline__ int padded(int k) { return (k + 127) & ~127; }      // whole ring items

__device__ __forceinline__ float4 load4(const float* p, int n) {       // elements from n on read as zero
    if (n >= 4 && (reinterpret_cast<uintptr_t>(p) & 15) == 0) return *reinterpret_cast<const float4*>(p);
    return make_float4(n > 0 ? p[0] : 0.f, n > 1 ? p[1] : 0.f, n > 2 ? p[2] : 0.f, n > 3 ? p[3] : 0.f);
}

constexpr int kKept = 4;                // quads of a vector that a thread keeps in registers

// The norm scales of a product's input, requested before the wait for the kernel before it (they are constant).
struct StagedScales {
    float4 s1[kKept], s2[kKept];
    __device__ __forceinline__ void request(const RowsArgs& a) {
        if (a.pro == PRO_CONCAT) return;
        const float* second = a.pro == PRO_POST_NORM ? a.b1 : a.s2;
#pragma unroll
        for (int i = 0; i < kKept; ++i) {
            const int j = (threadIdx.x + i * kThreads) * 4;
            s1[i] = load4(a.s1 + j, a.ka - j);          // zero beyond the end
            if (second) s2[i] = load4(second + j, a.ka - j);
        }
    }
};

// x + LayerNorm(x2) * s1 + b1, and - with s2 - LayerNorm(that) * s2 + b2
template <class Put> __device__ __forceinline__ void stage_post_norm(const RowsArgs& a, const StagedScales& sc, float* scratch, Put put) {
    const int step = kThreads * 4, j0 = threadIdx.x * 4, quads = (padded(a.ka) + step - 1) / step;
    float4 y[kKept], x[kKept];
#pragma unroll
    for (int i = 0; i < kKept; ++i) {
        const int j = j0 + i * step;
        y[i] = load4(a.x2 + j, a.ka - j);
        x[i] = load4(a.x + j, a.ka - j);
    }
    auto total = [](const float4& w) { return (w.x + w.y) + (w.z + w.w); };
    auto square = [&](float q, const float4& w, int j, float mean) {
        if (j < a.ka) q = fmaf(w.x - mean, w.x - mean, q);
        if (j + 1 < a.ka) q = fmaf(w.y - mean, w.y - mean, q);
        if (j + 2 < a.ka) q = fmaf(w.z - mean, w.z - mean, q);
        if (j + 3 < a.ka) q = fmaf(w.w - mean, w.w - mean, q);
        return q;
    };
    float s = 0.f, q = 0.f;
#pragma unroll
    for (int i = 0; i < kKept; ++i) s += total(y[i]);
    for (int i = kKept; i < quads; ++i) s += total(load4(a.x2 + j0 + i * step, a.ka - (j0 + i * step)));
    const float mean = lm::block_sum(s, scratch) / (float)a.ka;
#pragma unroll
    for (int i = 0; i < kKept; ++i) q = square(q, y[i], j0 + i * step, mean);
    for (int i = kKept; i < quads; ++i) q = square(q, load4(a.x2 + j0 + i * step, a.ka - (j0 + i * step)), j0 + i * step, mean);
    const float rstd = 1.0f / sqrtf(lm::block_sum(q, scratch) / (float)a.ka + a.eps);
    auto sum = [&](const float4& x, const float4& y, const float4& g, const float4& b) {
        return make_float4(x.x + fmaf((y.x - mean) * rstd, g.x, b.x), x.y + fmaf((y.y - mean) * rstd, g.y, b.y), x.z + fmaf((y.z - mean) * rstd, g.z, b.z),
                           x.w + fmaf((y.w - mean) * rstd, g.w, b.w));
    };
    auto late = [&](int j) { return sum(load4(a.x + j, a.ka - j), load4(a.x2 + j, a.ka - j), load4(a.s1 + j, a.ka - j), load4(a.b1 + j, a.ka - j)); };
#pragma unroll
    for (int i = 0; i < kKept; ++i) x[i] = sum(x[i], y[i], sc.s1[i], sc.s2[i]);       // zero beyond the end: scale and shift are
    if (a.x_out && blockIdx.x == 0) {
        auto store = [&](const float4& w, int j) {
            if (j < a.ka) a.x_out[j] = w.x;
            if (j + 1 < a.ka) a.x_out[j + 1] = w.y;
            if (j + 2 < a.ka) a.x_out[j + 2] = w.z;
            if (j + 3 < a.ka) a.x_out[j + 3] = w.w;
        };
#pragma unroll
        for (int i = 0; i < kKept; ++i) store(x[i], j0 + i * step);
        for (int i = kKept; i < quads; ++i) store(late(j0 + i * step), j0 + i * step);
    }
    float mean2 = 0.f, rstd2 = 1.f;
    if (a.s2) {
        s = q = 0.f;
#pragma unroll
        for (int i = 0; i < kKept; ++i) s += total(x[i]);
        for (int i = kKept; i < quads; ++i) s += total(late(j0 + i * step));
        mean2 = lm::block_sum(s, scratch) / (float)a.ka;
#pragma unroll
        for (int i = 0; i < kKept; ++i) q = square(q, x[i], j0 + i * step, mean2);
        for (int i = kKept; i < quads; ++i) q = square(q, late(j0 + i * step), j0 + i * step, mean2);
        rstd2 = 1.0f / sqrtf(lm::block_sum(q, scratch) / (float)a.ka + a.eps);
    }
    auto emit = [&](float4 w, int j) {
        if (j >= padded(a.ka)) return;
        if (a.s2) {
            const float4 g = load4(a.s2 + j, a.ka - j), b = a.b2 ? load4(a.b2 + j, a.ka - j) : make_float4(0.f, 0.f, 0.f, 0.f);
            w = make_float4(fmaf((w.x - mean2) * rstd2, g.x, b.x), fmaf((w.y - mean2) * rstd2, g.y, b.y), fmaf((w.z - mean2) * rstd2, g.z, b.z),
                            fmaf((w.w - mean2) * rstd2, g.w, b.w));
        }
        put(0, j, w);
    };
#pragma unroll
    for (int i = 0; i < kKept; ++i) emit(x[i], j0 + i * step);
    for (int i = kKept; i < quads; ++i) emit(late(j0 + i * step), j0 + i * step);
}

// The input vectors of a product, normalised or gated, four elements at a time: put(piece, j, values); zeros from the end of a
// vector to its padded length.
template <class Put> __device__ __forceinline__ void stage_input(const RowsArgs& a, const StagedScales& sc, float* scratch, Put put) {
    const int step = kThreads * 4, j0 = threadIdx.x * 4;
    if (a.pro == PRO_POST_NORM) {
        stage_post_norm(a, sc, scratch, put);
        return;
    }
    if (a.pro == PRO_LAYER_NORM || a.pro == PRO_RMS) {
        float4 v[kKept];
#pragma unroll
        for (int i = 0; i < kKept; ++i) v[i] = load4(a.x + j0 + i * step, a.ka - (j0 + i * step));
        auto quad = [&](int i) { return i < kKept ? v[i] : load4(a.x + j0 + i * step, a.ka - (j0 + i * step)); };
        const int quads = (padded(a.ka) + step - 1) / step;
        float mean = 0.f;
        if (a.pro == PRO_LAYER_NORM) {
            float s = 0.f;
#pragma unroll
            for (int i = 0; i < kKept; ++i) s += (v[i].x + v[i].y) + (v[i].z + v[i].w);
            for (int i = kKept; i < quads; ++i) {
                const float4 w = quad(i);
                s += (w.x + w.y) + (w.z + w.w);
            }
            mean = lm::block_sum(s, scratch) / (float)a.ka;
        }
        float q = 0.f;
        auto square = [&](const float4& w, int j) {
            if (j < a.ka) q = fmaf(w.x - mean, w.x - mean, q);
            if (j + 1 < a.ka) q = fmaf(w.y - mean, w.y - mean, q);
            if (j + 2 < a.ka) q = fmaf(w.z - mean, w.z - mean, q);
            if (j + 3 < a.ka) q = fmaf(w.w - mean, w.w - mean, q);
        };
#pragma unroll
        for (int i = 0; i < kKept; ++i) square(v[i], j0 + i * step);
        for (int i = kKept; i < quads; ++i) square(quad(i), j0 + i * step);
        const float rstd = 1.0f / sqrtf(lm::block_sum(q, scratch) / (float)a.ka + a.eps);
        auto emit = [&](const float4& w, int j, const float4& s1, const float4& s2) {
            if (j >= padded(a.ka)) return;
            const float x = (w.x - mean) * rstd, y = (w.y - mean) * rstd, z = (w.z - mean) * rstd, t = (w.w - mean) * rstd;
            const float4 b = a.b1 ? load4(a.b1 + j, a.ka - j) : make_float4(0.f, 0.f, 0.f, 0.f);
            put(0, j, make_float4(fmaf(x, s1.x, b.x), fmaf(y, s1.y, b.y), fmaf(z, s1.z, b.z), fmaf(t, s1.w, b.w)));
            if (a.s2) put(1, j, make_float4(x * s2.x, y * s2.y, z * s2.z, t * s2.w));
        };
#pragma unroll
        for (int i = 0; i < kKept; ++i) emit(v[i], j0 + i * step, sc.s1[i], sc.s2[i]);
        for (int i = kKept; i < quads; ++i) {
            const int j = j0 + i * step;
            emit(quad(i), j, load4(a.s1 + j, a.ka - j), a.s2 ? load4(a.s2 + j, a.ka - j) : make_float4(0.f, 0.f, 0.f, 0.f));
        }
        return;                                         // both pieces come from the norm
    }
    if (a.pro == PRO_GATED_RMS) {
        float4 v[kKept];
        float q = 0.f;
        auto square = [&](const float4& w) { q += (w.x * w.x + w.y * w.y) + (w.z * w.z + w.w * w.w); };
#pragma unroll
        for (int i = 0; i < kKept; ++i) {
            v[i] = load4(a.x + j0 + i * step, a.ka - (j0 + i * step));
            square(v[i]);
        }
        for (int j = j0 + kKept * step; j < a.ka; j += step) square(load4(a.x + j, a.ka - j));
        const float rstd = 1.0f / sqrtf(lm::block_sum(q, scratch) / (float)a.ka + a.eps);
        auto emit = [&](const float4& w, int j, const float4& s) {
            if (j >= padded(a.ka)) return;
            const float4 g = load4(a.gate + j, a.ka - j);
            put(0, j, make_float4(w.x * rstd * s.x * g.x, w.y * rstd * s.y * g.y, w.z * rstd * s.z * g.z, w.w * rstd * s.w * g.w));
        };
#pragma unroll
        for (int i = 0; i < kKept; ++i) emit(v[i], j0 + i * step, sc.s1[i]);
        for (int j = j0 + kKept * step; j < padded(a.ka); j += step) emit(load4(a.x + j, a.ka - j), j, load4(a.s1 + j, a.ka - j));
    } else {
#pragma unroll 4
        for (int j = j0; j < padded(a.ka); j += step) {
            if (a.split) {
                auto at = [&](int i) { return i >= a.ka ? 0.f : i < a.split ? a.x[i] : a.x2[i - a.split]; };
                put(0, j, make_float4(at(j), at(j + 1), at(j + 2), at(j + 3)));
            } else {
                put(0, j, load4(a.x + j, a.ka - j));
            }
        }
    }
#pragma unroll 4
    for (int j = j0; j < padded(a.kb); j += step) put(1, j, load4(a.x2 + j, a.kb - j));
}

__device__ __forceinline__ void finish_row(const RowsArgs& a, int row, float v) {
    if (row >= a.na) return;
    if (a.epi == EPI_MIXER_IN) {
        if (row < a.n_silu) v = lm::silu(v);
        else if (row >= a.n_sigmoid) v = lm::sigmoid(v);
    } else if (a.epi == EPI_RESIDUAL) {
        v = fmaf(a.alpha, v, a.resid[row]);
    } else if (a.epi == EPI_BIAS) {
        v += a.bias[row];
    } else if (a.epi == EPI_RELU_SQUARED) {
        v = v > 0.f ? v * v : 0.f;
    } else if (a.epi == EPI_SOFTCAP) {
        v = a.alpha * tanhf(v / a.alpha);
    }
    a.out[row] = v;
}

// Any type and row length: two rows per unit in FFMA, a team of warps splitting the columns.
template <class T>
__global__ void __launch_bounds__(kThreads) rows_kernel(const RowsArgs a) {
    rcu_kernel_entry();
    extern __shared__ __align__(16) float xs[];        // input A, input B
    __shared__ float scratch[32];
    __shared__ float red[kWarps][kRows];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int parts = a.parts, teams = kWarps / parts, team = warp / parts, part = warp % parts;
    const int ua = (a.na + kRows - 1) / kRows, units = ua + (a.dual ? 0 : a.pairs);
    const int xb = padded(a.ka);
    StagedScales sc;
    sc.request(a);
    stage_input(a, sc, scratch, [&](int piece, int j, const float4& v) { *reinterpret_cast<float4*>(xs + (piece ? xb : 0) + j) = v; });
    if (a.C > 0 && blockIdx.x == 0) append_latent<T>(a, scratch);
    __syncthreads();
    const T *wa = reinterpret_cast<const T*>(a.wa), *wb = reinterpret_cast<const T*>(a.wb);
    for (int u = team * gridDim.x + blockIdx.x; u < units; u += gridDim.x * teams) {
        float acc[kRows] = {};
        auto dot = [&](const T* w0, const T* w1, const float* x, int K) {
#pragma unroll 8
            for (int k = part * 32 + lane; k < K; k += parts * 32) {
                acc[0] = fmaf(to_f32<T>(w0[k]), x[k], acc[0]);
                acc[1] = fmaf(to_f32<T>(w1[k]), x[k], acc[1]);
            }
        };
        const size_t r0 = (size_t)u * kRows, r1 = min(u * kRows + 1, a.na - 1);
        if (a.dual || u < ua) dot(wa + r0 * a.ka, wa + r1 * a.ka, xs, a.ka);
        if (a.dual) dot(wb + r0 * a.kb, wb + r1 * a.kb, xs + xb, a.kb);
        else if (u >= ua) dot(wb + (size_t)(u - ua) * a.kb, wb + (size_t)(u - ua + a.pairs) * a.kb, xs + xb, a.kb);
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
                finish_row(a, u * kRows, acc[0]);
                finish_row(a, u * kRows + 1, acc[1]);
            } else {
                a.out2[u - ua] = lm::gelu_tanh(acc[0]) * acc[1];
            }
        }
    }
}

// bf16 weights, rows of whole 64-element blocks.  A unit is sixteen rows of piece A (or of both pieces, dual), or eight gate and
// their eight up rows.  ma / mb: [columns within a block, row, block] maps of the pieces, box 64 x 8 x 2.
__global__ void __launch_bounds__(kThreads) rows_mma_kernel(const __grid_constant__ CUtensorMap ma, const __grid_constant__ CUtensorMap mb,
                                                            const __grid_constant__ RowsArgs a) {
    extern __shared__ unsigned char smem_dyn[];        // rings (1024-byte aligned), then the inputs in fragment order
    __shared__ float scratch[32];
    __shared__ float red[2][kWarps][kUnit];
    __shared__ __align__(8) uint64_t full[kWarps][kMaxSlots];
    __shared__ volatile int abort_flag;
    unsigned char* rings = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_dyn) + 1023) & ~(uintptr_t)1023);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int slots = a.slots, parts = a.parts, teams = kWarps / parts, team = warp / parts, part = warp % parts;
    unsigned char* ring = rings + (size_t)warp * slots * kSlotBytes;
    // Input element k as columns 0 (rounding) and 1 (remainder) of a 16 x 8 operand: lane 4 n + (k % 8) / 2 of block k / 16 holds it
    uint32_t* xf = reinterpret_cast<uint32_t*>(rings + (size_t)kWarps * slots * kSlotBytes);
    const int xb = padded(a.ka);                        // one word per element
    const int ua = (a.na + kUnit - 1) / kUnit, units = ua + (a.dual ? 0 : (a.pairs + kUnit / 2 - 1) / (kUnit / 2));
    const int ia = (a.ka + kItem - 1) / kItem, ib = (a.kb + kItem - 1) / kItem;      // items of a piece
    const int gt = team * gridDim.x + blockIdx.x, gteams = gridDim.x * teams;      // a last, partial round of units spreads over the SMs
    auto items_of = [&](int u) { return a.dual ? ia + ib : (u < ua ? ia : ib); };
    int pu = gt, pi = part, pslot = 0;                  // next item to request: unit, item, slot
    auto request = [&]() {
        const bool pair = !a.dual && pu >= ua, b = pair || (a.dual && pi >= ia);
        const CUtensorMap* map = b ? &mb : &ma;
        const int block = 2 * (a.dual && b ? pi - ia : pi), row = pair ? (pu - ua) * (kUnit / 2) : pu * kUnit;
        unsigned char* dst = ring + pslot * kSlotBytes;
        uint64_t* bar = &full[warp][pslot];
        if (pi < items_of(pu)) {
            gemvq8::mbar_expect_tx(bar, kSlotBytes);
            gemvq8::tma_load_3d(dst, map, 0, row, block, bar);
            gemvq8::tma_load_3d(dst + kSlotBytes / 2, map, 0, pair ? row + a.pairs : row + kUnit / 2, block, bar);
        } else {
            gemvq8::mbar_arrive(bar);                   // a warp with no item in a unit passes through it with an empty slot
        }
        if (++pslot == slots) pslot = 0;
        pi += parts;
        if (pi >= items_of(pu)) {
            pu += gteams;
            pi = part;
        }
    };

    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    if (threadIdx.x == 0) abort_flag = 0;
    if (lane == 0) {
        for (int i = 0; i < slots; ++i) gemvq8::mbar_init(&full[warp][i], 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        for (int i = 0; i < slots && pu < units; ++i) request();
    }
    __syncwarp();
    StagedScales sc;
    sc.request(a);
    asm volatile("griddepcontrol.wait;" ::: "memory");

    stage_input(a, sc, scratch, [&](int piece, int j, const float4& v) {
        uint32_t h0, l0, h1, l1;
        lm::split2(v.x, v.y, h0, l0);
        lm::split2(v.z, v.w, h1, l1);
        uint32_t* f = xf + (piece ? xb : 0) + (j >> 4) * 16 + ((j & 7) >> 1) * 2 + ((j >> 3) & 1);
        f[0] = h0; f[2] = h1;                           // column 0, lanes t and t + 1
        f[8] = l0; f[10] = l1;                          // column 1
    });
    if (a.C > 0 && blockIdx.x == 0) append_latent<__nv_bfloat16>(a, scratch);
    __syncthreads();

    const int row = lane & 7;
    const uint32_t frag = lm::smem_addr(ring) + ((lane >> 3) & 1) * (kSlotBytes / 2) + row * 128;
    uint32_t sw[4];                                     // swizzled place of this lane's 16 bytes in each 16-column step of a block
#pragma unroll
    for (int i = 0; i < 4; ++i) sw[i] = (uint32_t)(((2 * i + (lane >> 4)) ^ row) << 4);
    bool ok = true;
    int slot = 0, parity = 0;
    uint32_t phase = 0;
    for (int u = gt; u < units; u += gteams, parity ^= 1) {
        const int n = items_of(u);
        float c0[4] = {}, c1[4] = {};
        int i = part;
        do {
            // once a wait has given up, the warp only keeps its team's barriers company
            ok = ok && gemvq8::mbar_wait_spin(&full[warp][slot], phase, &abort_flag, a.status);
            if (ok && i < n) {
                const bool b = a.dual ? i >= ia : u >= ua;
                const uint2* xv = reinterpret_cast<const uint2*>(xf + (b ? xb : 0) + (a.dual && b ? i - ia : i) * kItem) + lane;
                const uint32_t base = frag + slot * kSlotBytes;
#pragma unroll
                for (int s = 0; s < kItem / 16; ++s) {
                    uint32_t w[4];
                    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                                 : "=r"(w[0]), "=r"(w[1]), "=r"(w[2]), "=r"(w[3])
                                 : "r"(base + (s >> 2) * 1024 + sw[s & 3]));
                    uint2 x = make_uint2(0u, 0u);
                    if (lane < 8) x = xv[s * 8];
                    if (s & 1) lm::mma(c1, w, x.x, x.y);
                    else lm::mma(c0, w, x.x, x.y);
                }
            }
            __syncwarp();                               // every lane has read the slot
            if (lane == 0 && ok && pu < units) request();
            if (ok && ++slot == slots) { slot = 0; phase ^= 1; }
            i += parts;
        } while (i < n);
        // lanes 4 g: columns 0 and 1 of rows g and g + 8
        float lo = (c0[0] + c1[0]) + (c0[1] + c1[1]), hi = (c0[2] + c1[2]) + (c0[3] + c1[3]);
        int g = lane >> 2;
        bool mine = (lane & 3) == 0;
        if (parts > 1) {
            if (mine) {
                red[parity][warp][g] = lo;
                red[parity][warp][g + 8] = hi;
            }
            asm volatile("bar.sync %0, %1;" ::"r"(1 + team), "r"(parts * 32) : "memory");
            mine = part == 0 && lane < 8;
            g = lane;
            if (mine) {
                lo = hi = 0.f;
                for (int q = 0; q < parts; ++q) {
                    lo += red[parity][team * parts + q][g];
                    hi += red[parity][team * parts + q][g + 8];
                }
            }
        }
        if (mine) {
            if (a.dual || u < ua) {
                finish_row(a, u * kUnit + g, lo);
                finish_row(a, u * kUnit + g + 8, hi);
            } else {
                const int p = (u - ua) * (kUnit / 2) + g;
                if (p < a.pairs) a.out2[p] = lm::gelu_tanh(lo) * hi;
            }
        }
    }
    if (!ok) {
        // A wait gave up (the status word says so).  Before leaving, give this warp's copies in flight another chance to land.
        for (int i = 0; i < slots; ++i)
            for (int t = 0; t < (1 << 16) && !gemvq8::mbar_test_wait(&full[warp][i], i < slot ? phase ^ 1 : phase); ++t) {}
    }
}

// [64 columns, rows, K / 64 blocks] view of a row-major bf16 matrix
bool make_block_map(CUtensorMap* map, const void* base, uint64_t rows, uint64_t K) {
    gemvq8::EncodeTiledFn fn = gemvq8::encode_tiled_fn();
    if (!fn) return false;
    cuuint64_t dims[3] = {64, rows, K / 64};
    cuuint64_t strides[2] = {K * 2, 128};
    cuuint32_t box[3] = {64, kUnit / 2, kItem / 64};
    cuuint32_t estr[3] = {1, 1, 1};
    return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
              CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

// (cos, sin) of the step's position for one frequency table
struct AngleTable {
    const float* freqs;
    float2* out;
    int pairs;
    float magnitude;
};

// x0 = x = embedding row of the token; an id outside the table is clamped and flagged.  The last n_angles CTAs fill an angle table each.
template <class T>
__global__ void __launch_bounds__(kThreads) embed_kernel(const int32_t* token, const T* __restrict__ table, int vocab, int width, float* x0, float* x,
                                                         const AngleTable* __restrict__ angles, int n_angles, const uint32_t* d_pos, int* status) {
    rcu_kernel_entry();
    const int rows = (int)gridDim.x - n_angles;
    if ((int)blockIdx.x >= rows) {
        const AngleTable t = angles[blockIdx.x - rows];
        for (int i = threadIdx.x; i < t.pairs; i += kThreads) t.out[i] = lm::rotary_angle(t.freqs, t.pairs, i, *d_pos, t.magnitude);
        return;
    }
    int t = *token;
    if (t < 0 || t >= vocab) {
        if (threadIdx.x == 0 && blockIdx.x == 0) atomicOr(status, RCU_DEVFLAG_BOUNDS);
        t = t < 0 ? 0 : vocab - 1;
    }
    for (int j = blockIdx.x * kThreads + threadIdx.x; j < width; j += rows * kThreads) {
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
        constexpr int kAhead = 16;            // rows requested before the first of them is written back
        for (int d0 = g; d0 < D; d0 += kWarps * kAhead) {
            float s[kAhead];
#pragma unroll
            for (int i = 0; i < kAhead; ++i) s[i] = d0 + i * kWarps < D ? S[(size_t)(d0 + i * kWarps) * E + e] : 0.f;
#pragma unroll
            for (int i = 0; i < kAhead; ++i) {
                const int d = d0 + i * kWarps;
                if (d >= D) break;
                s[i] = fmaf(dec, s[i], k[d] * v);
                S[(size_t)d * E + e] = s[i];
                o = fmaf(q[d], s[i], o);
            }
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

__device__ __forceinline__ void load8(const float* p, float (&v)[8]) {
    *reinterpret_cast<float4*>(v) = *reinterpret_cast<const float4*>(p);
    *reinterpret_cast<float4*>(v + 4) = *reinterpret_cast<const float4*>(p + 4);
}

// row pitch of the partial results: C sums, the maximum and the sum of the weights, in whole 16 bytes
__host__ __device__ __forceinline__ int partial_pitch(int C) { return ((C + 3) & ~3) + 4; }

// Attention of one token over the cached latents: CTA = (run of positions, eight heads), a warp per head.  Positions are
// staged kSub at a time in shared memory (rows padded with zeros to a multiple of eight elements) and shared by the heads; a
// lane owns eight consecutive features of every 256.  Each warp keeps an online softmax and its share of the weighted
// latents.  partial[split][head]: C sums, then the maximum and the sum of the weights.  PW: 256-feature groups of a row.
template <class T, int PW>
__global__ void __launch_bounds__(kThreads) latent_step_kernel(const float* __restrict__ qa, const T* __restrict__ ring, int ring_rows, int window,
                                                               const uint32_t* d_pos, float* __restrict__ partial, int H, int C, int R) {
    rcu_kernel_entry();
    extern __shared__ __align__(16) float q_s[];         // [kHeads][WP], then the staged rows [kSub][WP]
    const int W = C + R, WP = (W + 7) & ~7, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    T* rows = reinterpret_cast<T*>(q_s + (size_t)kHeads * WP);
    const int h0 = blockIdx.y * kHeads, h = h0 + warp;
    const int pos = (int)*d_pos, first = max(0, pos - window + 1), n = pos - first + 1;
    const int per = (n + gridDim.x - 1) / gridDim.x;
    const int begin = first + min(n, (int)blockIdx.x * per), end = first + min(n, ((int)blockIdx.x + 1) * per);
    constexpr int VEC = 16 / (int)sizeof(T);
    const bool vec = W % VEC == 0;
    if (h < H)
        for (int c = lane; c < WP; c += 32) q_s[warp * WP + c] = c < W ? qa[(size_t)h * W + c] : 0.f;
    for (int i = threadIdx.x; i < kSub * (WP - W); i += kThreads) rows[(i / (WP - W)) * WP + W + i % (WP - W)] = from_f32<T>(0.f);
    __syncwarp();
    float q[PW][8], o[PW][8];
#pragma unroll
    for (int g = 0; g < PW; ++g) {
        const int c = g * 256 + lane * 8;
#pragma unroll
        for (int e = 0; e < 8; ++e) q[g][e] = o[g][e] = 0.f;
        if (c < WP && h < H) load8(q_s + warp * WP + c, q[g]);
    }
    float m = -INFINITY, l = 0.f;
    for (int p0 = begin; p0 < end; p0 += kSub) {
        const int np = min(kSub, end - p0);
        __syncthreads();
        for (int r = warp; r < np; r += kWarps) {
            const T* src = ring + (size_t)((p0 + r) % ring_rows) * W;
            if (vec)
                for (int c = lane * VEC; c < W; c += 32 * VEC) *reinterpret_cast<uint4*>(rows + r * WP + c) = *reinterpret_cast<const uint4*>(src + c);
            else
                for (int c = lane; c < W; c += 32) rows[r * WP + c] = src[c];
        }
        __syncthreads();
        if (h >= H) continue;
        float s[kSub];
        float mt = -INFINITY;
#pragma unroll
        for (int r = 0; r < kSub; ++r) {
            s[r] = 0.f;
            if (r < np) {
#pragma unroll
                for (int g = 0; g < PW; ++g) {
                    const int c = g * 256 + lane * 8;
                    if (c < WP) {
                        float v[8];
                        load8(rows + r * WP + c, v);
#pragma unroll
                        for (int e = 0; e < 8; ++e) s[r] = fmaf(q[g][e], v[e], s[r]);
                    }
                }
            }
        }
#pragma unroll
        for (int r = 0; r < kSub; ++r) {
            s[r] = r < np ? warp_sum(s[r]) : -INFINITY;
            mt = fmaxf(mt, s[r]);
        }
        const float mn = fmaxf(m, mt), corr = expf(m - mn);
        l *= corr;
#pragma unroll
        for (int g = 0; g < PW; ++g)
#pragma unroll
            for (int e = 0; e < 8; ++e) o[g][e] *= corr;
        m = mn;
#pragma unroll
        for (int r = 0; r < kSub; ++r) {
            if (r >= np) break;
            const float p = expf(s[r] - mn);
            l += p;
#pragma unroll
            for (int g = 0; g < PW; ++g) {
                const int c = g * 256 + lane * 8;
                if (c < C) {
                    float v[8];
                    load8(rows + r * WP + c, v);
#pragma unroll
                    for (int e = 0; e < 8; ++e) o[g][e] = fmaf(p, v[e], o[g][e]);
                }
            }
        }
    }
    if (h >= H) return;
    float* dst = partial + ((size_t)blockIdx.x * H + h) * partial_pitch(C);
#pragma unroll
    for (int g = 0; g < PW; ++g)
#pragma unroll
        for (int e = 0; e < 8; ++e) {
            const int c = g * 256 + lane * 8 + e;
            if (c < C) dst[c] = o[g][e];
        }
    if (lane == 0) {
        dst[partial_pitch(C) - 2] = m;
        dst[partial_pitch(C) - 1] = l;
    }
}

// The same for bf16 rings, on the tensor cores: CTA = (run of positions, sixteen heads).  Per sixteen positions: scores as
// [heads, features] . [features, positions], the features split over the warps and summed in shared memory; online softmax, a
// thread per (head, position); the weighted latents as [heads, positions] . [positions, features], each warp owning a run
// of features.  Queries and weights enter as bf16 value plus remainder.
constexpr int kMmaHeads = 16;
template <int PC>
__global__ void __launch_bounds__(kThreads) latent_step_mma_kernel(const float* __restrict__ qa, const lm::bf16* __restrict__ ring, int ring_rows, int window,
                                                                   const uint32_t* d_pos, float* __restrict__ partial, int H, int C, int R) {
    rcu_kernel_entry();
    using lm::bf16;
    extern __shared__ __align__(16) bf16 tiles[];        // queries (value, remainder), staged rows
    __shared__ float part[kWarps][kMmaHeads][kSub + 1];
    __shared__ __align__(16) bf16 ph[kMmaHeads][kSub + 8], pl[kMmaHeads][kSub + 8];
    __shared__ float corr_s[kMmaHeads];
    const int W = C + R, wp = (W + 15) & ~15, ld = wp + 8;
    bf16 *qh = tiles, *ql = qh + kMmaHeads * ld, *rows = ql + kMmaHeads * ld;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
    const int h0 = blockIdx.y * kMmaHeads;
    const int pos = (int)*d_pos, first = max(0, pos - window + 1), n = pos - first + 1;
    const int per = (n + gridDim.x - 1) / gridDim.x;
    const int begin = first + min(n, (int)blockIdx.x * per), end = first + min(n, ((int)blockIdx.x + 1) * per);
    auto stage = [&](int p0) {
        const int np = min(kSub, end - p0), octets = wp / 8;
        if (W % 8 == 0) {
#pragma unroll 6
            for (int i = threadIdx.x; i < kSub * octets; i += kThreads) {
                const int r = i / octets, c = (i - r * octets) * 8;
                const bool in = r < np && c < W;
                lm::cp_async16(rows + r * ld + c, ring + (in ? (size_t)((p0 + r) % ring_rows) * W + c : 0), in);
            }
            lm::cp_commit();
        } else {
            for (int i = threadIdx.x; i < kSub * wp; i += kThreads) {
                const int r = i / wp, c = i - r * wp;
                rows[r * ld + c] = r < np && c < W ? ring[(size_t)((p0 + r) % ring_rows) * W + c] : __float2bfloat16_rn(0.f);
            }
        }
    };
    if (begin < end) stage(begin);
    const int quads = wp / 4;
#pragma unroll 8
    for (int i = threadIdx.x; i < kMmaHeads * quads; i += kThreads) {
        const int r = i / quads, c = (i - r * quads) * 4;
        const float4 v = h0 + r < H ? load4(qa + (size_t)(h0 + r) * W + c, W - c) : make_float4(0.f, 0.f, 0.f, 0.f);
        uint2 hi, lo;
        lm::split2(v.x, v.y, hi.x, lo.x);
        lm::split2(v.z, v.w, hi.y, lo.y);
        *reinterpret_cast<uint2*>(qh + r * ld + c) = hi;
        *reinterpret_cast<uint2*>(ql + r * ld + c) = lo;
    }
    const int sh = threadIdx.x >> 4, sp = threadIdx.x & 15;              // this thread's (head, position) of the softmax
    float m = -INFINITY, l = 0.f, o[PC][2][4];
#pragma unroll
    for (int c = 0; c < PC; ++c)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[c][0][e] = o[c][1][e] = 0.f;
    for (int p0 = begin; p0 < end; p0 += kSub) {
        if (p0 != begin) {
            __syncthreads();
            stage(p0);
        }
        lm::cp_wait<0>();
        __syncthreads();
        float s0[4] = {}, s1[4] = {};
        for (int k0 = warp * 16; k0 < wp; k0 += kWarps * 16) {
            uint32_t ah[4], al[4], b[4];
            lm::load_a(ah, qh, ld, 0, k0);
            lm::load_a(al, ql, ld, 0, k0);
            lm::load_b(b, rows, ld, 0, k0);
            lm::mma(s0, ah, b[0], b[1]);
            lm::mma(s1, ah, b[2], b[3]);
            lm::mma(s0, al, b[0], b[1]);
            lm::mma(s1, al, b[2], b[3]);
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            part[warp][g + (e >> 1) * 8][2 * t + (e & 1)] = s0[e];
            part[warp][g + (e >> 1) * 8][8 + 2 * t + (e & 1)] = s1[e];
        }
        __syncthreads();
        float s = 0.f;
#pragma unroll
        for (int w = 0; w < kWarps; ++w) s += part[w][sh][sp];
        if (p0 + sp >= end) s = -INFINITY;
        float mt = s;
#pragma unroll
        for (int x = 8; x > 0; x >>= 1) mt = fmaxf(mt, __shfl_xor_sync(0xffffffffu, mt, x));
        const float mn = fmaxf(m, mt), corr = expf(m - mn), p = expf(s - mn);
        float ps = p;
#pragma unroll
        for (int x = 8; x > 0; x >>= 1) ps += __shfl_xor_sync(0xffffffffu, ps, x);
        l = l * corr + ps;
        m = mn;
        const bf16 hi = __float2bfloat16_rn(p);
        ph[sh][sp] = hi;
        pl[sh][sp] = __float2bfloat16_rn(p - __bfloat162float(hi));
        if (sp == 0) corr_s[sh] = corr;
        __syncthreads();
        uint32_t ah[4], al[4];
        lm::load_a(ah, &ph[0][0], kSub + 8, 0, 0);
        lm::load_a(al, &pl[0][0], kSub + 8, 0, 0);
        const float c0 = corr_s[g], c1 = corr_s[g + 8];
#pragma unroll
        for (int c = 0; c < PC; ++c) {
            const int col = (warp + c * kWarps) * 16;
            if (col >= wp) break;
            uint32_t b[4];
            lm::load_b_t(b, rows, ld, col, 0);
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                o[c][x][0] *= c0; o[c][x][1] *= c0;
                o[c][x][2] *= c1; o[c][x][3] *= c1;
                lm::mma(o[c][x], ah, b[2 * x], b[2 * x + 1]);
                lm::mma(o[c][x], al, b[2 * x], b[2 * x + 1]);
            }
        }
    }
    const int pitch = partial_pitch(C);
    float* dst = partial + ((size_t)blockIdx.x * H + h0) * pitch;
#pragma unroll
    for (int c = 0; c < PC; ++c)
#pragma unroll
        for (int x = 0; x < 2; ++x)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int col = (warp + c * kWarps) * 16 + 8 * x + 2 * t + (e & 1), r = g + (e >> 1) * 8;
                if (col < C && h0 + r < H) dst[(size_t)r * pitch + col] = o[c][x][e];
            }
    if (sp == 0 && h0 + sh < H) {
        dst[(size_t)sh * pitch + pitch - 2] = m;
        dst[(size_t)sh * pitch + pitch - 1] = l;
    }
}

// Merge of a head's partial results and its values: out[h] = W_uv[h] . (weighted latent).  CTA = (head, run of value rows).
// Groups of threads merge different splits, four features per thread and load.
template <class T>
__global__ void __launch_bounds__(kThreads) latent_values_kernel(const float* __restrict__ partial, int splits, const T* __restrict__ uv, float* __restrict__ out,
                                                                 int H, int C, int E, int rows_per) {
    extern __shared__ __align__(16) float c_s[];        // [groups][quads * 4], the sum in group 0
    __shared__ float wgt[kMaxSplits];
    const int h = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int pitch = partial_pitch(C), quads = (C + 3) / 4, groups = max(1, kThreads / quads);
    // the warp's first two rows of up to 1024 features are requested before the wait (weights are constant)
    constexpr int VEC = 16 / (int)sizeof(T), kEarly = 1024 / (32 * VEC);
    const bool vec = C % VEC == 0 && C <= 1024 && (reinterpret_cast<uintptr_t>(uv) & 15) == 0;
    const int e0 = blockIdx.y * rows_per + warp, e1 = min(E, ((int)blockIdx.y + 1) * rows_per);
    uint4 early[2][kEarly];
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    if (vec) {
#pragma unroll
        for (int r = 0; r < 2; ++r)
#pragma unroll
            for (int i = 0; i < kEarly; ++i) {
                const int e = e0 + r * kWarps, c = (lane + 32 * i) * VEC;
                if (e < e1 && c < C) early[r][i] = ld_stream_v4(uv + ((size_t)h * E + e) * C + c);
            }
    }
    asm volatile("griddepcontrol.wait;" ::: "memory");
    const float* ph = partial + (size_t)h * pitch;
    const size_t stride = (size_t)H * pitch;
    if (warp == 0) {
        const float m0 = lane < splits ? ph[lane * stride + pitch - 2] : -INFINITY, m1 = lane + 32 < splits ? ph[(lane + 32) * stride + pitch - 2] : -INFINITY;
        const float l0 = lane < splits ? ph[lane * stride + pitch - 1] : 0.f, l1 = lane + 32 < splits ? ph[(lane + 32) * stride + pitch - 1] : 0.f;
        const float M = warp_max(fmaxf(m0, m1));
        const float w0 = lane < splits ? expf(m0 - M) : 0.f, w1 = lane + 32 < splits ? expf(m1 - M) : 0.f;
        const float l = warp_sum(w0 * l0 + w1 * l1);
        wgt[lane] = w0 / l;
        wgt[lane + 32] = w1 / l;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < groups * quads; i += kThreads) {
        const int g = i / quads, c = (i - g * quads) * 4;
        float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 16
        for (int j = g; j < splits; j += groups) {
            const float4 v = *reinterpret_cast<const float4*>(ph + j * stride + c);
            s.x = fmaf(wgt[j], v.x, s.x);
            s.y = fmaf(wgt[j], v.y, s.y);
            s.z = fmaf(wgt[j], v.z, s.z);
            s.w = fmaf(wgt[j], v.w, s.w);
        }
        *reinterpret_cast<float4*>(c_s + (size_t)g * quads * 4 + c) = s;
    }
    __syncthreads();
    for (int c = threadIdx.x; c < C; c += kThreads) {
        float s = c_s[c];
        for (int g = 1; g < groups; ++g) s += c_s[(size_t)g * quads * 4 + c];
        c_s[c] = s;
    }
    __syncthreads();
    for (int r = 0; e0 + r * kWarps < e1; ++r) {
        const int e = e0 + r * kWarps;
        const T* w = uv + ((size_t)h * E + e) * C;
        float acc = 0.f;
        if (vec) {
#pragma unroll
            for (int i = 0; i < kEarly; ++i) {
                const int c = (lane + 32 * i) * VEC;
                if (c < C) {
                    uint4 raw = r == 0 ? early[0][i] : early[1][i];
                    if (r > 1) raw = ld_stream_v4(w + c);
                    const T* wv = reinterpret_cast<const T*>(&raw);
#pragma unroll
                    for (int x = 0; x < VEC; ++x) acc = fmaf(to_f32<T>(wv[x]), c_s[c + x], acc);
                }
            }
        } else {
            for (int c = lane; c < C; c += 32) acc = fmaf(to_f32<T>(w[c]), c_s[c], acc);
        }
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
#pragma unroll 8
        for (int i = threadIdx.x; i < n; i += 1024) {
            const float v = logits[i];
            if (v > best || idx == 0x7fffffff) { best = v; idx = i; }
        }
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
    float *x0, *xa, *xb, *mix, *act, *y, *sub, *q, *qa, *partial, *logits;
    float *angle_pool, *angle_tables, *arrived;      // (cos, sin) pairs; AngleTable[n_angles]; counters of the grouped attention
    std::vector<float2*> run_angles;                 // per run: its pairs (null: no grouped mixer)
    int n_angles = 0;
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

uint64_t grouped_seen(const rcu_stack_run& r) {      // rows a token can see at most
    const uint64_t most = r.chunk ? r.chunk : r.window ? r.window : r.ring_rows;
    return std::min<uint64_t>(most, r.ring_rows);
}
int grouped_splits(const rcu_device* dev, const rcu_stack_run& r, int dt) {
    const bool mma = gstep::takes_mma(dt, (int)r.dim, (int)r.vdim, r.state);
    const int groups = gstep::head_groups((int)r.heads, (int)r.kv_heads, mma ? gstep::kMmaHeads : gstep::kFmaHeads);
    return gstep::splits(dev->sm_count, (int)r.kv_heads * groups, grouped_seen(r), mma);
}

// Warps per team.  A CTA's time is bound below by the memory system (its units' items, one after the other) and by the longest
// chain of items a warp works through, an item taking a warp about twice as long as the memory system; ending a unit
// (reduction, epilogue) counts as an item, and meeting the team's other warps as another.
int plan_parts(int grid, int units, int items) {
    int best = 1;
    double best_cost = -1.0;
    const double stream = (double)((units + grid - 1) / grid) * items;
    for (int parts = 1; parts <= kWarps; parts *= 2) {
        const long long teams = (long long)grid * (kWarps / parts), rounds = (units + teams - 1) / teams;
        const double chain = 2.0 * rounds * ((items + parts - 1) / parts + (parts > 1 ? 2 : 1));
        const double cost = std::max(stream, chain) + 0.25 * chain;
        if (best_cost < 0.0 || cost < best_cost) { best = parts; best_cost = cost; }
    }
    return best;
}

template <class T> rcu_status launch_rows(rcu_device* dev, RowsArgs a) {
    a.status = dev->d_status;
    const bool has_b = a.kb > 0 && a.wb;
    const size_t inputs = ((size_t)padded(a.ka) + (size_t)padded(a.kb)) * 4, per_slot = (size_t)kWarps * kSlotBytes;
    const size_t most = (size_t)dev->smem_optin - 4096;
    // Rings as deep as shared memory allows: bytes in flight are worth more than room for the next kernel's CTA (measured with
    // rings held to half an SM: 414 us per token against 376 at width 2048).
    a.slots = inputs + 1024 < most ? (int)std::min<size_t>(kMaxSlots, (most - 1024 - inputs) / per_slot) : 0;
    const bool blocks = sizeof(T) == 2 && a.ka % 64 == 0 && (!has_b || a.kb % 64 == 0) && a.slots >= 2 &&
                        ((reinterpret_cast<uintptr_t>(a.wa) | reinterpret_cast<uintptr_t>(a.wb)) & 15) == 0;
    if (blocks) {
        const int units = (a.na + kUnit - 1) / kUnit + (a.dual ? 0 : (a.pairs + kUnit / 2 - 1) / (kUnit / 2));
        const int ia = (a.ka + kItem - 1) / kItem, ib = has_b ? (a.kb + kItem - 1) / kItem : 0;
        a.parts = plan_parts(dev->sm_count, units, a.dual ? ia + ib : std::max(ia, ib));
        const int grid = std::max(1, std::min(dev->sm_count, units));
        CUtensorMap ma, mb;
        if (!make_block_map(&ma, a.wa, a.na, a.ka) || !make_block_map(&mb, has_b ? a.wb : a.wa, has_b ? (a.dual ? a.na : 2 * a.pairs) : a.na, has_b ? a.kb : a.ka))
            return rcu_fail(dev, RCU_ERR_CUDA, "stack: cuTensorMapEncodeTiled failed (%d x %d)", a.na, a.ka);
        RCU_CUDA(dev, cudaFuncSetAttribute(rows_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)most));
        RCU_CUDA(dev, rcu_launch(dev, rows_mma_kernel, grid, kThreads, 1024 + a.slots * per_slot + inputs, ma, mb, a));
    } else {
        const int units = (a.na + kRows - 1) / kRows + (a.dual ? 0 : a.pairs), nca = (a.ka + 255) / 256, ncb = (a.kb + 255) / 256;
        a.parts = plan_parts(dev->sm_count, units, a.dual ? nca + ncb : std::max(nca, ncb));
        const int teams = kWarps / a.parts, grid = std::max(1, std::min(4 * dev->sm_count, (units + teams - 1) / teams));
        if (inputs > most) return rcu_fail(dev, RCU_ERR_UNSUPPORTED, "stack: input vectors of %d + %d do not fit shared memory", a.ka, a.kb);
        RCU_CUDA(dev, cudaFuncSetAttribute(rows_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)most));
        RCU_CUDA(dev, rcu_launch(dev, rows_kernel<T>, grid, kThreads, inputs, a));
    }
    RCU_LAUNCH_CHECK(dev);
    return RCU_OK;
}

rcu_status launch_latent_step(rcu_device* dev, const rcu_stack* s, const rcu_stack_run& r, int dt) {
    const int H = (int)r.heads, C = (int)r.kv_rank, R = (int)r.rot_dim, splits = latent_splits(r);
#define RCU_LS(KERN_, GRID_, T_)                                                                                                                 \
    do {                                                                                                                                         \
        RCU_CUDA(dev, cudaFuncSetAttribute(KERN_, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)std::max(smem, (size_t)(48 * 1024))));       \
        RCU_CUDA(dev, rcu_launch(dev, KERN_, GRID_, kThreads, smem, s->qa, (const T_*)r.state, (int)r.ring_rows, (int)r.window, s->d_pos, s->partial, H, C, R)); \
    } while (0)
    if (dt == RCU_BF16) {
        const int wp = (C + R + 15) & ~15;
        const size_t smem = (size_t)(2 * kMmaHeads + kSub) * (wp + 8) * sizeof(lm::bf16);
        const dim3 grid(splits, (H + kMmaHeads - 1) / kMmaHeads);
        if (wp <= 256) RCU_LS(latent_step_mma_kernel<2>, grid, lm::bf16);
        else if (wp <= 640) RCU_LS(latent_step_mma_kernel<5>, grid, lm::bf16);
        else RCU_LS(latent_step_mma_kernel<10>, grid, lm::bf16);
    } else {
        const int WP = (C + R + 7) & ~7;
        const size_t smem = (size_t)kHeads * WP * 4 + (size_t)kSub * WP * sizeof(float);
        const dim3 grid(splits, (H + kHeads - 1) / kHeads);
        switch ((WP + 255) / 256) {
            case 1: RCU_LS((latent_step_kernel<float, 1>), grid, float); break;
            case 2: RCU_LS((latent_step_kernel<float, 2>), grid, float); break;
            case 3: RCU_LS((latent_step_kernel<float, 3>), grid, float); break;
            case 4: RCU_LS((latent_step_kernel<float, 4>), grid, float); break;
            default: RCU_LS((latent_step_kernel<float, 5>), grid, float); break;
        }
    }
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
    RCU_CUDA(dev, rcu_launch(dev, embed_kernel<T>, (W + kThreads - 1) / kThreads + s->n_angles, kThreads, 0, token, (const T*)s->embed, (int)c.vocab, W, s->x0, x,
                             (const AngleTable*)s->angle_tables, s->n_angles, s->d_pos, dev->d_status));
    RCU_LAUNCH_CHECK(dev);
    const float *after = nullptr, *after_shift = nullptr;      // post-norm layers: the norm that awaits the last sublayer's output
    // the residual stream as a product's input; with a sublayer output waiting, the sum goes to the other stream buffer
    auto stream_input = [&](RowsArgs& a) {
        a.ka = W;
        a.x = x;
        a.eps = c.eps;
        a.pro = PRO_CONCAT;
        if (after) {
            a.pro = PRO_POST_NORM; a.x2 = s->sub; a.s1 = after; a.b1 = after_shift; a.x_out = other;
            std::swap(x, other);
        }
    };
    for (size_t k = 0; k < s->runs.size(); ++k) {
        const rcu_stack_run& r = s->runs[k];
        if (c.layer == RCU_LAYER_POST_NORM) {
            const int H = (int)r.heads, G = (int)r.kv_heads, D = (int)r.dim, E = (int)r.vdim;
            RowsArgs in = {};
            stream_input(in);
            in.wa = r.mix_in; in.na = (H + G) * D + G * E; in.epi = r.mix_bias ? EPI_BIAS : EPI_STORE; in.bias = (const float*)r.mix_bias; in.out = s->mix;
            STACK_TRY(launch_rows<T>(dev, in));
            const gstep::Args at{s->mix, (const float*)r.mix_norm, (const float*)r.kv_norm, s->run_angles[k], (const float*)r.sink, r.state, s->d_pos, s->y, s->partial,
                                 (uint32_t*)s->arrived, H, G, D, E, (int)r.rot_pairs, (int)r.ring_rows,
                                 r.window ? (int)std::min<uint32_t>(r.window, 1u << 30) : 1 << 30, (int)std::min<uint32_t>(r.chunk, 1u << 30), c.eps, r.scale};
            STACK_TRY(gstep::launch(dev, c.weight_dt, at, grouped_splits(dev, r, c.weight_dt)));
            RowsArgs o = {};
            o.wa = r.out; o.na = W; o.ka = H * E; o.pro = PRO_CONCAT; o.x = s->y; o.out = s->sub;
            o.epi = r.out_bias ? EPI_BIAS : EPI_STORE; o.bias = (const float*)r.out_bias;
            STACK_TRY(launch_rows<T>(dev, o));
            after = (const float*)r.norm1; after_shift = (const float*)r.norm1_shift;
            if (r.ff) {
                RowsArgs up = {};
                stream_input(up);
                up.wa = r.gate_up; up.na = (int)r.ff; up.epi = EPI_RELU_SQUARED; up.out = s->act;
                STACK_TRY(launch_rows<T>(dev, up));
                RowsArgs down = {};
                down.wa = r.down; down.na = W; down.ka = (int)r.ff; down.pro = PRO_CONCAT; down.x = s->act; down.out = s->sub;
                STACK_TRY(launch_rows<T>(dev, down));
                after = (const float*)r.norm2; after_shift = (const float*)r.norm2_shift;
            }
            continue;
        }
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
            STACK_TRY(launch_latent_step(dev, s, r, c.weight_dt));
            const int per = 2 * kWarps, quads = (C + 3) / 4, groups = std::max(1, kThreads / quads);
            RCU_CUDA(dev, rcu_launch(dev, latent_values_kernel<T>, dim3(H, (E + per - 1) / per), kThreads, (size_t)groups * quads * 16, s->partial, latent_splits(r),
                                     (const T*)r.ukv + (size_t)H * D * C, s->y, H, C, E, per));
            RCU_LAUNCH_CHECK(dev);
            out.pro = PRO_CONCAT; out.x = s->y;
        }
        STACK_TRY(launch_rows<T>(dev, out));
    }
    RowsArgs head = {};
    if (after) {
        stream_input(head);
        head.x_out = nullptr;
        head.s2 = s->final_norm; head.b2 = (const float*)c.final_shift;
    } else {
        head.ka = W; head.pro = PRO_LAYER_NORM; head.x = x; head.s1 = s->final_norm; head.b1 = (const float*)c.final_shift; head.eps = c.eps;
    }
    head.wa = s->head; head.na = (int)c.vocab; head.out = logits;
    if (c.logit_softcap > 0.f) { head.epi = EPI_SOFTCAP; head.alpha = c.logit_softcap; }
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
    RCU_REQUIRE(dev, cfg->layer == RCU_LAYER_PARALLEL || cfg->layer == RCU_LAYER_POST_NORM, "stack: unknown kind of layer %d", cfg->layer);
    const bool post = cfg->layer == RCU_LAYER_POST_NORM;
    size_t mix = 0, act = 1, y = 0, q = 1, qa = 1, partial = 1, arrived = 1, pairs = 1;
    std::vector<int> table_of(cfg->n_runs, -1);
    std::vector<uint32_t> table_run;                 // the run each angle table comes from
    for (uint32_t i = 0; i < cfg->n_runs; ++i) {
        const rcu_stack_run& r = runs[i];
        if (post != (r.mixer == RCU_MIXER_GROUPED))
            return rcu_fail(dev, RCU_ERR_UNSUPPORTED, "stack: run %u: post-norm layers take grouped heads, parallel ones the other mixers", i);
        RCU_REQUIRE(dev, r.norm1 && r.mix_in && r.mix_norm && r.out && r.state && r.heads && r.dim && r.vdim, "stack: run %u lacks a weight or a size", i);
        RCU_REQUIRE(dev, r.ff == 0 || (r.norm2 && r.gate_up && r.down), "stack: run %u lacks a feed-forward weight", i);
        RCU_REQUIRE(dev, r.heads <= 65535, "stack: run %u has too many heads", i);
        RCU_REQUIRE(dev, !post || (r.norm1_shift && (r.ff == 0 || r.norm2_shift) && !r.enter), "stack: run %u lacks a norm's shift, or enters a pass", i);
        if (r.mixer == RCU_MIXER_LIGHTNING) {
            RCU_REQUIRE(dev, r.decay, "stack: run %u has no decay", i);
            mix = std::max(mix, (size_t)r.heads * 2 * (r.dim + r.vdim));
        } else if (r.mixer == RCU_MIXER_GROUPED) {
            RCU_REQUIRE(dev, r.kv_heads && r.heads % r.kv_heads == 0 && r.kv_norm && (r.rot_pairs == 0 || r.freqs) && 2 * r.rot_pairs <= r.dim && r.ring_rows,
                        "stack: run %u lacks a weight or a size", i);
            if (r.dim > 1024 || r.vdim > 512) return rcu_fail(dev, RCU_ERR_UNSUPPORTED, "stack: run %u: heads of %u and %u (at most 1024 and 512)", i, r.dim, r.vdim);
            mix = std::max(mix, (size_t)(r.heads + r.kv_heads) * r.dim + (size_t)r.kv_heads * r.vdim);
            partial = std::max(partial, (size_t)grouped_splits(dev, r, cfg->weight_dt) * r.heads * gstep::pitch_of((int)r.vdim));
            arrived = std::max(arrived, (size_t)r.heads);
            for (size_t t = 0; t < table_run.size() && table_of[i] < 0; ++t) {
                const rcu_stack_run& o = runs[table_run[t]];
                if (o.freqs == r.freqs && o.rot_pairs == r.rot_pairs && o.rot_magnitude == r.rot_magnitude) table_of[i] = (int)t;
            }
            if (table_of[i] < 0) {
                table_of[i] = (int)table_run.size();
                table_run.push_back(i);
            }
            pairs = std::max(pairs, (size_t)r.rot_pairs);
        } else {
            RCU_REQUIRE(dev, r.mixer == RCU_MIXER_LATENT, "stack: run %u has an unknown mixer", i);
            RCU_REQUIRE(dev, r.q_rank && r.kv_rank && r.kv_norm && r.uq && r.ukv && (r.rot_pairs == 0 || r.freqs) && 2 * r.rot_pairs <= r.rot_dim,
                        "stack: run %u lacks a weight or a size", i);
            RCU_REQUIRE(dev, r.window > 0 && r.ring_rows > 0, "stack: run %u has no window", i);
            if (r.kv_rank + r.rot_dim > 1280) return rcu_fail(dev, RCU_ERR_UNSUPPORTED, "stack: cached rows of %u (at most 1280)", r.kv_rank + r.rot_dim);
            mix = std::max(mix, (size_t)r.q_rank + r.kv_rank + r.rot_dim);
            q = std::max(q, (size_t)r.heads * (r.dim + r.rot_dim));
            qa = std::max(qa, (size_t)r.heads * (r.kv_rank + r.rot_dim));
            partial = std::max(partial, (size_t)latent_splits(r) * r.heads * partial_pitch((int)r.kv_rank));
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
    const size_t n_tables = table_run.size();
    const size_t sizes[] = {cfg->width, cfg->width, cfg->width, mix, act, y, cfg->width, q, qa, partial, 2 * pairs * n_tables, n_tables * (sizeof(AngleTable) / 4), arrived};
    float** ptrs[] = {&s->x0, &s->xa, &s->xb, &s->mix, &s->act, &s->y, &s->sub, &s->q, &s->qa, &s->partial, &s->angle_pool, &s->angle_tables, &s->arrived};
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
    std::vector<AngleTable> tables;
    for (size_t t = 0; t < n_tables; ++t) {
        const rcu_stack_run& r = runs[table_run[t]];
        tables.push_back(AngleTable{(const float*)r.freqs, (float2*)s->angle_pool + t * pairs, (int)r.rot_pairs, r.rot_magnitude});
    }
    for (uint32_t i = 0; i < cfg->n_runs; ++i) s->run_angles.push_back(table_of[i] < 0 ? nullptr : tables[table_of[i]].out);
    s->n_angles = (int)n_tables;
    if (n_tables) st = rcu_h2d(dev, s->angle_tables, tables.data(), n_tables * sizeof(AngleTable));
    if (st == RCU_OK) st = rcu_memset(dev, s->arrived, 0, arrived * 4);
    if (st == RCU_OK) st = rcu_sync(dev);             // the tables' host copy ends with this call
    if (st == RCU_OK) st = rcu_stack_set_position(s, 0);
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
    {
        const uint64_t seen = r.mixer == RCU_MIXER_GROUPED && r.chunk ? r.chunk : r.mixer == RCU_MIXER_GROUPED && !r.window ? ~0ull : r.window;
        RCU_REQUIRE(dev, r.mixer == RCU_MIXER_LIGHTNING || r.ring_rows >= seen || s->position < r.ring_rows, "stack: the cache is full (%u rows)", r.ring_rows);
    }
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
