// RMSNorm of one attention head followed by the rotation of its leading interleaved pairs, by a power-of-two group of lanes:
// shared by the query and key paths of prompts (stream_ops.cu, grouped_attention.cu).
#pragma once
#include "lm_math.cuh"

namespace lm {

struct HeadNorm {
    const float* scale;        // [dim], shared by the heads
    const float* angles;       // [tokens, 2 pairs]: (cos, sin) of a pair side by side
    int dim, pairs;
    float eps;
};

// lanes of a group that hold a head, V consecutive elements each
__host__ __device__ __forceinline__ int head_lanes(int dim, int V) {
    int n = 1;
    while (n * V < dim && n < 32) n *= 2;
    return n;
}

template <class T, int V> struct alignas(sizeof(T) * V) HeadVec { T v[V]; };

// V > 1: dim is a multiple of V and at most 32 V, every row starts on V elements; `s` is the lane's place in its group of `lanes`.
// V == 1: any dim, the group is the warp.  All lanes of the warp take part; `live` lanes store (second may be null: a second copy).
template <class T, int V>
__device__ __forceinline__ void head_norm_rotate(const HeadNorm& a, const T* x, const float2* cs, T* out, T* second, int s, int lanes, bool live) {
    if (V > 1) {
        const int c = s * V;
        const bool in = live && c < a.dim;
        float v[V];
        float q = 0.f;
        HeadVec<T, V> raw;
        if (in) raw = *reinterpret_cast<const HeadVec<T, V>*>(x + c);
#pragma unroll
        for (int e = 0; e < V; ++e) {
            v[e] = in ? to_f32<T>(raw.v[e]) : 0.f;
            q = fmaf(v[e], v[e], q);
        }
        for (int o = lanes >> 1; o > 0; o >>= 1) q += __shfl_xor_sync(0xffffffffu, q, o);
        const float rstd = 1.0f / sqrtf(q / (float)a.dim + a.eps);
        if (!in) return;
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] *= rstd * a.scale[c + e];
#pragma unroll
        for (int e = 0; e + 1 < V; e += 2) {
            const int i = (c + e) >> 1;
            if (i < a.pairs) {
                const float2 r = cs[i];
                const float u = v[e], w = v[e + 1];
                v[e] = u * r.x - w * r.y;
                v[e + 1] = w * r.x + u * r.y;
            }
        }
#pragma unroll
        for (int e = 0; e < V; ++e) raw.v[e] = from_f32<T>(v[e]);
        *reinterpret_cast<HeadVec<T, V>*>(out + c) = raw;
        if (second) *reinterpret_cast<HeadVec<T, V>*>(second + c) = raw;
    } else {
        float q = 0.f;
        for (int d = s; live && d < a.dim; d += 32) q = fmaf(to_f32<T>(x[d]), to_f32<T>(x[d]), q);
        const float rstd = 1.0f / sqrtf(warp_sum(q) / (float)a.dim + a.eps);
        if (!live) return;
        auto put = [&](int d, float v) {
            out[d] = from_f32<T>(v);
            if (second) second[d] = out[d];
        };
        for (int i = s; i < a.pairs; i += 32) {
            const float u = to_f32<T>(x[2 * i]) * (rstd * a.scale[2 * i]), w = to_f32<T>(x[2 * i + 1]) * (rstd * a.scale[2 * i + 1]);
            put(2 * i, u * cs[i].x - w * cs[i].y);
            put(2 * i + 1, w * cs[i].x + u * cs[i].y);
        }
        for (int d = 2 * a.pairs + s; d < a.dim; d += 32) put(d, to_f32<T>(x[d]) * (rstd * a.scale[d]));
    }
}

}  // namespace lm
