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

// V consecutive features of a head, one lane's part.  What a token's heads share is loaded once: dim is a multiple of V (V even) and at
// most 32 V, `s` the lane's place in its group of `lanes`.
template <class T, int V> struct HeadPart {
    float scale[V];
    float2 cs[V / 2];          // (1, 0) for features that are not rotated
    int c;
    bool in;

    __device__ __forceinline__ void load(const HeadNorm& a, long long token, int s, bool live) {
        c = s * V;
        in = live && c < a.dim;
        const int i0 = c / 2;
        const float2* angles = reinterpret_cast<const float2*>(a.angles) + token * a.pairs;
#pragma unroll
        for (int e = 0; e < V; e += 4) *reinterpret_cast<float4*>(scale + e) = in ? *reinterpret_cast<const float4*>(a.scale + c + e) : make_float4(0.f, 0.f, 0.f, 0.f);
        if (in && i0 + V / 2 <= a.pairs && a.pairs % 2 == 0) {
#pragma unroll
            for (int i = 0; i < V / 2; i += 2) *reinterpret_cast<float4*>(cs + i) = *reinterpret_cast<const float4*>(angles + i0 + i);
        } else {
#pragma unroll
            for (int i = 0; i < V / 2; ++i) cs[i] = in && i0 + i < a.pairs ? angles[i0 + i] : make_float2(1.f, 0.f);
        }
    }
    // all lanes of the group take part
    __device__ __forceinline__ HeadVec<T, V> apply(const HeadNorm& a, const HeadVec<T, V>& raw, int lanes) const {
        float v[V], q = 0.f;
#pragma unroll
        for (int e = 0; e < V; ++e) {
            v[e] = to_f32<T>(raw.v[e]);
            q = fmaf(v[e], v[e], q);
        }
        for (int o = lanes >> 1; o > 0; o >>= 1) q += __shfl_xor_sync(0xffffffffu, q, o);
        const float rstd = 1.0f / sqrtf(q / (float)a.dim + a.eps);
        HeadVec<T, V> out;
#pragma unroll
        for (int e = 0; e < V; e += 2) {
            const float u = v[e] * (rstd * scale[e]), w = v[e + 1] * (rstd * scale[e + 1]);
            out.v[e] = from_f32<T>(u * cs[e / 2].x - w * cs[e / 2].y);
            out.v[e + 1] = from_f32<T>(w * cs[e / 2].x + u * cs[e / 2].y);
        }
        return out;
    }
};

// Any dim, a warp per head; all lanes take part, `live` ones store (second may be null: a second copy).
template <class T>
__device__ __forceinline__ void head_norm_rotate(const HeadNorm& a, const T* x, long long token, T* out, T* second, int lane, bool live) {
    const float2* cs = reinterpret_cast<const float2*>(a.angles) + token * a.pairs;
    float q = 0.f;
    for (int d = lane; live && d < a.dim; d += 32) q = fmaf(to_f32<T>(x[d]), to_f32<T>(x[d]), q);
    const float rstd = 1.0f / sqrtf(warp_sum(q) / (float)a.dim + a.eps);
    if (!live) return;
    auto put = [&](int d, float v) {
        out[d] = from_f32<T>(v);
        if (second) second[d] = out[d];
    };
    for (int i = lane; i < a.pairs; i += 32) {
        const float u = to_f32<T>(x[2 * i]) * (rstd * a.scale[2 * i]), w = to_f32<T>(x[2 * i + 1]) * (rstd * a.scale[2 * i + 1]);
        put(2 * i, u * cs[i].x - w * cs[i].y);
        put(2 * i + 1, w * cs[i].x + u * cs[i].y);
    }
    for (int d = 2 * a.pairs + lane; d < a.dim; d += 32) put(d, to_f32<T>(x[d]) * (rstd * a.scale[d]));
}

}  // namespace lm
