// Row operations between the projections of a model that keeps its residual stream, norms and gates in 32 bits while
// its matrix products take 16-bit operands: norms of f32 rows (or of a column window of them) into any float type with an
// optional sigmoid gate, a sublayer's normalised output added to the stream, the gated activation of a feed-forward, and rotary
// positions on interleaved pairs with an explicit frequency table (alone, or behind a norm of each head).
#include <cmath>

#include "head_norm.cuh"

namespace {

struct NormArgs {
    const float* x;
    long long x_pitch;
    const float *scale, *shift;     // shift: nullable, added after the scale
    const void* gate;          // nullable: output *= sigmoid(gate[row * gate_pitch + j])
    long long gate_pitch;
    int N;
    float eps;
    int layer;                 // 1: LayerNorm, 0: RMSNorm
    __device__ __forceinline__ float affine(float v, int j) const { return shift ? fmaf(v, scale[j], shift[j]) : v * scale[j]; }
};

template <class G> __device__ __forceinline__ float gate_of(const NormArgs& a, size_t row, int j) {
    return lm::sigmoid(to_f32<G>(reinterpret_cast<const G*>(a.gate)[row * a.gate_pitch + j]));
}

// A warp per row, the row in registers (N <= 32 * PER).  The variance is the mean of the squared deviations, taken in
// a second pass over the registers.
template <class Out, int PER>
__global__ void __launch_bounds__(256) norm_rows_warp_kernel(const NormArgs a, Out* __restrict__ out, long long rows) {
    rcu_kernel_entry();
    const int lane = threadIdx.x & 31;
    const long long row = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (row >= rows) return;
    const float* xr = a.x + row * a.x_pitch;
    float v[PER];
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int j = lane + 32 * i;
        v[i] = j < a.N ? xr[j] : 0.f;
        s += v[i];
    }
    const float mean = a.layer ? warp_sum(s) / (float)a.N : 0.f;
    float q = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int j = lane + 32 * i;
        v[i] -= mean;
        if (j < a.N) q = fmaf(v[i], v[i], q);
    }
    const float rstd = 1.0f / sqrtf(warp_sum(q) / (float)a.N + a.eps);
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int j = lane + 32 * i;
        if (j < a.N) {
            float y = a.affine(v[i] * rstd, j);
            if (a.gate) y *= gate_of<Out>(a, (size_t)row, j);
            out[(size_t)row * a.N + j] = from_f32<Out>(y);
        }
    }
}

// A CTA per row of at most 256 * 4 * QUADS elements that starts on 16 bytes: the row in registers, four elements per load.
template <class Out, int QUADS>
__global__ void __launch_bounds__(256) norm_rows_quad_kernel(const NormArgs a, Out* __restrict__ out) {
    rcu_kernel_entry();
    __shared__ float scratch[32];
    const size_t row = blockIdx.x;
    const float* xr = a.x + row * a.x_pitch;
    float v[QUADS][4];
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < QUADS; ++i) {
        const int j = (threadIdx.x + i * 256) * 4;
        float4 q = make_float4(0.f, 0.f, 0.f, 0.f);
        if (j < a.N) q = *reinterpret_cast<const float4*>(xr + j);
        v[i][0] = q.x; v[i][1] = q.y; v[i][2] = q.z; v[i][3] = q.w;
        s += (q.x + q.y) + (q.z + q.w);
    }
    const float mean = a.layer ? lm::block_sum(s, scratch) / (float)a.N : 0.f;
    float q = 0.f;
#pragma unroll
    for (int i = 0; i < QUADS; ++i)
        if ((threadIdx.x + i * 256) * 4 < a.N)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                v[i][e] -= mean;
                q = fmaf(v[i][e], v[i][e], q);
            }
    const float rstd = 1.0f / sqrtf(lm::block_sum(q, scratch) / (float)a.N + a.eps);
    struct alignas(sizeof(Out) * 4) Quad { Out v[4]; };
#pragma unroll
    for (int i = 0; i < QUADS; ++i) {
        const int j = (threadIdx.x + i * 256) * 4;
        if (j >= a.N) continue;
        const float4 g = *reinterpret_cast<const float4*>(a.scale + j);
        float y[4] = {v[i][0] * rstd * g.x, v[i][1] * rstd * g.y, v[i][2] * rstd * g.z, v[i][3] * rstd * g.w};
        if (a.shift) {
            const float4 b = *reinterpret_cast<const float4*>(a.shift + j);
            y[0] += b.x; y[1] += b.y; y[2] += b.z; y[3] += b.w;
        }
        if (a.gate) {
            const Quad t = *reinterpret_cast<const Quad*>(reinterpret_cast<const Out*>(a.gate) + row * a.gate_pitch + j);
#pragma unroll
            for (int e = 0; e < 4; ++e) y[e] *= lm::sigmoid(to_f32<Out>(t.v[e]));
        }
        Quad o;
#pragma unroll
        for (int e = 0; e < 4; ++e) o.v[e] = from_f32<Out>(y[e]);
        *reinterpret_cast<Quad*>(out + row * a.N + j) = o;
    }
}

// A CTA per row, the row in shared memory.
template <class Out>
__global__ void __launch_bounds__(256) norm_rows_kernel(const NormArgs a, Out* __restrict__ out) {
    rcu_kernel_entry();
    extern __shared__ float row_s[];
    __shared__ float scratch[32];
    const size_t row = blockIdx.x;
    const float* xr = a.x + row * a.x_pitch;
    float s = 0.f;
    for (int j = threadIdx.x; j < a.N; j += 256) {
        const float v = xr[j];
        row_s[j] = v;
        s += v;
    }
    const float mean = a.layer ? lm::block_sum(s, scratch) / (float)a.N : 0.f;
    float q = 0.f;
    for (int j = threadIdx.x; j < a.N; j += 256) {
        const float d = row_s[j] - mean;
        q = fmaf(d, d, q);
    }
    const float rstd = 1.0f / sqrtf(lm::block_sum(q, scratch) / (float)a.N + a.eps);
    for (int j = threadIdx.x; j < a.N; j += 256) {
        float y = a.affine((row_s[j] - mean) * rstd, j);
        if (a.gate) y *= gate_of<Out>(a, row, j);
        out[row * a.N + j] = from_f32<Out>(y);
    }
}

template <class Out>
rcu_status launch_norm_rows(rcu_device* dev, const NormArgs& a, void* out, uint64_t rows) {
    const unsigned warp_grid = (unsigned)((rows + 7) / 8);
    if (a.N <= 128) rcu_launch(dev, norm_rows_warp_kernel<Out, 4>, warp_grid, 256, 0, a, (Out*)out, (long long)rows);
    else if (a.N <= 512) rcu_launch(dev, norm_rows_warp_kernel<Out, 16>, warp_grid, 256, 0, a, (Out*)out, (long long)rows);
    else if (a.N % 4 == 0 && a.N <= 8192 && a.x_pitch % 4 == 0 && a.gate_pitch % 4 == 0 &&
             ((reinterpret_cast<uintptr_t>(a.x) | reinterpret_cast<uintptr_t>(a.scale) | reinterpret_cast<uintptr_t>(a.shift) | reinterpret_cast<uintptr_t>(out)) & 15) == 0 &&
             (reinterpret_cast<uintptr_t>(a.gate) & (4 * sizeof(Out) - 1)) == 0) {
        if (a.N <= 1024) rcu_launch(dev, norm_rows_quad_kernel<Out, 1>, (unsigned)rows, 256, 0, a, (Out*)out);
        else if (a.N <= 2048) rcu_launch(dev, norm_rows_quad_kernel<Out, 2>, (unsigned)rows, 256, 0, a, (Out*)out);
        else if (a.N <= 4096) rcu_launch(dev, norm_rows_quad_kernel<Out, 4>, (unsigned)rows, 256, 0, a, (Out*)out);
        else rcu_launch(dev, norm_rows_quad_kernel<Out, 8>, (unsigned)rows, 256, 0, a, (Out*)out);
    } else {
        const size_t smem = (size_t)a.N * 4;
        if (smem + 1024 > (size_t)dev->smem_optin) return rcu_fail(dev, RCU_ERR_UNSUPPORTED, "norm_rows: rows of %d do not fit shared memory", a.N);
        if (smem > 40 * 1024) RCU_CUDA(dev, cudaFuncSetAttribute(norm_rows_kernel<Out>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        rcu_launch(dev, norm_rows_kernel<Out>, (unsigned)rows, 256, smem, a, (Out*)out);
    }
    RCU_LAUNCH_CHECK(dev);
    return RCU_OK;
}

template <class T, int V>
__global__ void __launch_bounds__(256) glu_kernel(const T* __restrict__ x, T* __restrict__ out, size_t n, int F, int act) {
    rcu_kernel_entry();
    struct alignas(sizeof(T) * V) Vec { T v[V]; };
    const int fv = F / V;
    for (size_t i = (size_t)blockIdx.x * 256 + threadIdx.x; i < n; i += (size_t)gridDim.x * 256) {
        const size_t row = i / fv, j = (i % fv) * V;
        const Vec g = *reinterpret_cast<const Vec*>(x + row * 2 * F + j), u = *reinterpret_cast<const Vec*>(x + row * 2 * F + F + j);
        Vec o;
#pragma unroll
        for (int e = 0; e < V; ++e) {
            const float z = to_f32<T>(g.v[e]);
            o.v[e] = from_f32<T>((act == RCU_GELU ? lm::gelu_tanh(z) : lm::silu(z)) * to_f32<T>(u.v[e]));
        }
        *reinterpret_cast<Vec*>(out + row * F + j) = o;
    }
}

template <class T> rcu_status launch_glu(rcu_device* dev, const void* x, void* out, uint64_t rows, uint64_t F, int act) {
    constexpr int V = 16 / (int)sizeof(T);
    const bool vec = F % V == 0 && ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
    const size_t n = vec ? rows * F / V : rows * F;
    const unsigned grid = (unsigned)grid_for(n, 256, dev->sm_count * 16);
    if (vec) rcu_launch(dev, glu_kernel<T, V>, grid, 256, 0, (const T*)x, (T*)out, n, (int)F, act);
    else rcu_launch(dev, glu_kernel<T, 1>, grid, 256, 0, (const T*)x, (T*)out, n, (int)F, act);
    RCU_LAUNCH_CHECK(dev);
    return RCU_OK;
}

// One CTA per token: the angles of its pairs once in shared memory, then every head.
template <class T>
__global__ void __launch_bounds__(128) rotary_kernel(const T* x, const float* __restrict__ freqs, T* out, int H, int D, int first, int pairs,
                                                     float magnitude, uint32_t position) {
    rcu_kernel_entry();
    extern __shared__ float2 cs[];
    const size_t t = blockIdx.x;
    for (int i = threadIdx.x; i < pairs; i += blockDim.x) cs[i] = lm::rotary_angle(freqs, pairs, i, position + (uint32_t)t, magnitude);
    __syncthreads();
    const T* xr = x + t * (size_t)H * D;
    T* orow = out + t * (size_t)H * D;
    for (int j = threadIdx.x; j < H * pairs; j += blockDim.x) {
        const int h = j / pairs, i = j % pairs;
        const size_t o = (size_t)h * D + first + 2 * i;
        const float u = to_f32<T>(xr[o]), v = to_f32<T>(xr[o + 1]);
        orow[o] = from_f32<T>(u * cs[i].x - v * cs[i].y);
        orow[o + 1] = from_f32<T>(v * cs[i].x + u * cs[i].y);
    }
    if (x != out)
        for (int j = threadIdx.x; j < H * D; j += blockDim.x) {
            const int d = j % D;
            if (d < first || d >= first + 2 * pairs) orow[j] = xr[j];
        }
}

// Rows of W values into stream rows of `pitch` f32 words: the values, then (pitch > W) their bf16 roundings.
template <class T>
__global__ void __launch_bounds__(256) stream_rows_kernel(const T* __restrict__ x, float* __restrict__ out, int W, int pitch) {
    rcu_kernel_entry();
    const size_t row = blockIdx.x;
    float* o = out + row * pitch;
    __nv_bfloat16* copy = reinterpret_cast<__nv_bfloat16*>(o + W);
    for (int j = threadIdx.x; j < W; j += 256) {
        const float v = to_f32<T>(x[row * W + j]);
        o[j] = v;
        if (pitch > W) copy[j] = __float2bfloat16_rn(v);
    }
}

struct PostNormArgs {
    const float *x, *y, *scale, *shift;
    float* out;                // rows as x's; may be x
    int W, pitch;
    float eps;
};

// out = x + LayerNorm(y) * scale + shift.  A CTA per row of at most 1024 * QUADS elements whose quads start on 16 bytes: the row in
// registers, the old stream requested together with it.
template <int QUADS>
__global__ void __launch_bounds__(256) post_norm_quad_kernel(const PostNormArgs a) {
    rcu_kernel_entry();
    __shared__ float scratch[32];
    const size_t row = blockIdx.x;
    const float *yr = a.y + row * a.W, *xr = a.x + row * a.pitch;
    float4 v[QUADS], x[QUADS];
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < QUADS; ++i) {
        const int j = (threadIdx.x + i * 256) * 4;
        v[i] = x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (j < a.W) {
            v[i] = *reinterpret_cast<const float4*>(yr + j);
            x[i] = *reinterpret_cast<const float4*>(xr + j);
        }
        s += (v[i].x + v[i].y) + (v[i].z + v[i].w);
    }
    const float mean = lm::block_sum(s, scratch) / (float)a.W;
    float q = 0.f;
#pragma unroll
    for (int i = 0; i < QUADS; ++i)
        if ((threadIdx.x + i * 256) * 4 < a.W) {
            v[i].x -= mean; v[i].y -= mean; v[i].z -= mean; v[i].w -= mean;
            q += (v[i].x * v[i].x + v[i].y * v[i].y) + (v[i].z * v[i].z + v[i].w * v[i].w);
        }
    const float rstd = 1.0f / sqrtf(lm::block_sum(q, scratch) / (float)a.W + a.eps);
    float* o = a.out + row * a.pitch;
    uint2* copy = reinterpret_cast<uint2*>(o + a.W);
#pragma unroll
    for (int i = 0; i < QUADS; ++i) {
        const int j = (threadIdx.x + i * 256) * 4;
        if (j >= a.W) continue;
        const float4 g = *reinterpret_cast<const float4*>(a.scale + j), b = *reinterpret_cast<const float4*>(a.shift + j);
        const float4 r = make_float4(x[i].x + fmaf(v[i].x * rstd, g.x, b.x), x[i].y + fmaf(v[i].y * rstd, g.y, b.y), x[i].z + fmaf(v[i].z * rstd, g.z, b.z),
                                     x[i].w + fmaf(v[i].w * rstd, g.w, b.w));
        *reinterpret_cast<float4*>(o + j) = r;
        if (a.pitch > a.W) {
            const __nv_bfloat162 lo = __floats2bfloat162_rn(r.x, r.y), hi = __floats2bfloat162_rn(r.z, r.w);
            copy[j / 4] = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
        }
    }
}

// Any width: a warp per row, three passes over it.
__global__ void __launch_bounds__(256) post_norm_kernel(const PostNormArgs a, long long rows) {
    rcu_kernel_entry();
    const int lane = threadIdx.x & 31;
    const long long row = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (row >= rows) return;
    const float *yr = a.y + row * a.W, *xr = a.x + row * a.pitch;
    float s = 0.f, q = 0.f;
    for (int j = lane; j < a.W; j += 32) s += yr[j];
    const float mean = warp_sum(s) / (float)a.W;
    for (int j = lane; j < a.W; j += 32) q = fmaf(yr[j] - mean, yr[j] - mean, q);
    const float rstd = 1.0f / sqrtf(warp_sum(q) / (float)a.W + a.eps);
    float* o = a.out + row * a.pitch;
    __nv_bfloat16* copy = reinterpret_cast<__nv_bfloat16*>(o + a.W);
    for (int j = lane; j < a.W; j += 32) {
        const float r = xr[j] + fmaf((yr[j] - mean) * rstd, a.scale[j], a.shift[j]);
        o[j] = r;
        if (a.pitch > a.W) copy[j] = __float2bfloat16_rn(r);
    }
}

__global__ void __launch_bounds__(128) rotary_angles_kernel(const float* __restrict__ freqs, float2* __restrict__ out, int pairs, float magnitude, uint32_t position,
                                                            long long n) {
    rcu_kernel_entry();
    const long long i = (long long)blockIdx.x * 128 + threadIdx.x;
    if (i < n) out[i] = lm::rotary_angle(freqs, pairs, (int)(i % pairs), position + (uint32_t)(i / pairs), magnitude);
}

constexpr int kHeadsPerGroup = 4;        // heads of a token that a group of lanes takes, their loads in flight together

// dst[t, h] = rotate(rms_norm(x[t, head h])); a group of lanes per (token, kHeadsPerGroup heads), or (V == 1) a warp per head
template <class T, int V>
__global__ void __launch_bounds__(256) norm_rotary_kernel(const lm::HeadNorm a, const T* __restrict__ x, long long pitch, T* __restrict__ out, int H, long long n,
                                                          int lanes) {
    rcu_kernel_entry();
    const int lane = threadIdx.x & 31;
    const long long item = ((long long)blockIdx.x * 8 + (threadIdx.x >> 5)) * (32 / lanes) + lane / lanes;
    const bool live = item < n;
    if constexpr (V == 1) {
        const long long t = live ? item / H : 0;
        const int h = live ? (int)(item - t * H) : 0;
        lm::head_norm_rotate<T>(a, x + t * pitch + (long long)h * a.dim, t, out + (t * H + h) * a.dim, (T*)nullptr, lane, live);
    } else {
        using Vec = lm::HeadVec<T, V>;
        constexpr int N = kHeadsPerGroup;
        const int per = (H + N - 1) / N;
        const long long t = live ? item / per : 0;
        const int h0 = live ? (int)(item - t * per) * N : 0;
        lm::HeadPart<T, V> part;
        part.load(a, t, lane & (lanes - 1), live);
        const T* src = x + t * pitch + (long long)h0 * a.dim + part.c;
        T* dst = out + (t * H + h0) * a.dim + part.c;
        Vec v[N];
#pragma unroll
        for (int j = 0; j < N; ++j) v[j] = part.in && h0 + j < H ? *reinterpret_cast<const Vec*>(src + (long long)j * a.dim) : Vec{};
#pragma unroll
        for (int j = 0; j < N; ++j) {
            const Vec y = part.apply(a, v[j], lanes);
            if (part.in && h0 + j < H) *reinterpret_cast<Vec*>(dst + (long long)j * a.dim) = y;
        }
    }
}

template <class T>
void launch_norm_rotary(rcu_device* dev, const lm::HeadNorm& a, const void* x, long long pitch, void* out, int H, long long T_) {
    constexpr int V = 16 / (int)sizeof(T), N = kHeadsPerGroup;
    const bool vec = a.dim % V == 0 && a.dim <= 32 * V && pitch % V == 0 &&
                     ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(a.scale) | reinterpret_cast<uintptr_t>(a.angles)) & 15) == 0;
    const long long n = vec ? T_ * ((H + N - 1) / N) : T_ * H;
    const int lanes = vec ? lm::head_lanes(a.dim, V) : 32, per = 8 * (32 / lanes);
    const unsigned grid = (unsigned)((n + per - 1) / per);
    if (vec) rcu_launch(dev, norm_rotary_kernel<T, V>, grid, 256, 0, a, (const T*)x, pitch, (T*)out, H, n, lanes);
    else rcu_launch(dev, norm_rotary_kernel<T, 1>, grid, 256, 0, a, (const T*)x, pitch, (T*)out, H, n, lanes);
}

}  // namespace

extern "C" {

rcu_status rcu_norm_rows(rcu_device* dev, int kind, const rcu_tensor* x, uint32_t x_col, const rcu_tensor* scale, const rcu_tensor* shift,
                         const rcu_tensor* gate, uint32_t gate_col, float eps, rcu_tensor* dst) {
    if (!dev) return RCU_ERR_INVALID_ARG;
    RCU_REQUIRE(dev, t_valid(x) && t_valid(scale) && t_valid(dst), "norm_rows: invalid tensor descriptor");
    RCU_REQUIRE(dev, kind == RCU_LAYER_NORM || kind == RCU_RMS_NORM, "norm_rows: LayerNorm or RMSNorm");
    RCU_REQUIRE(dev, x->dt == RCU_F32 && scale->dt == RCU_F32 && dt_is_float(dst->dt), "norm_rows: f32 input and scale, float output");
    const uint64_t N = t_numel(scale), pitch = x->shape[x->rank - 1], rows = t_numel(x) / pitch;
    RCU_REQUIRE(dev, x_col + N <= pitch && N <= 0x7fffffffull && rows <= 0x7fffffffull, "norm_rows: the columns lie outside the rows");
    RCU_REQUIRE(dev, t_numel(dst) == rows * N, "norm_rows: dst holds %llu elements, expected %llu", (unsigned long long)t_numel(dst), (unsigned long long)(rows * N));
    RCU_REQUIRE(dev, !shift || (t_valid(shift) && shift->dt == RCU_F32 && t_numel(shift) == N), "norm_rows: the shift is f32 of the scale's length");
    uint64_t gp = 0;
    if (gate) {
        RCU_REQUIRE(dev, t_valid(gate) && gate->dt == dst->dt, "norm_rows: the gate has the output's dtype");
        gp = gate->shape[gate->rank - 1];
        RCU_REQUIRE(dev, gate_col + N <= gp && t_numel(gate) / gp == rows, "norm_rows: the gate's columns lie outside its rows");
    }
    DevGuard g(dev->ordinal);
    NormArgs a{(const float*)x->data + x_col, (long long)pitch, (const float*)scale->data, shift ? (const float*)shift->data : nullptr,
               gate ? (const char*)gate->data + (size_t)gate_col * dt_esize(gate->dt) : nullptr, (long long)gp, (int)N, eps, kind == RCU_LAYER_NORM};
    switch (dst->dt) {
        case RCU_F32: return launch_norm_rows<float>(dev, a, dst->data, rows);
        case RCU_F16: return launch_norm_rows<__half>(dev, a, dst->data, rows);
        default: return launch_norm_rows<__nv_bfloat16>(dev, a, dst->data, rows);
    }
}

rcu_status rcu_glu(rcu_device* dev, int act, const rcu_tensor* x, rcu_tensor* dst) {
    if (!dev) return RCU_ERR_INVALID_ARG;
    RCU_REQUIRE(dev, t_valid(x) && t_valid(dst), "glu: invalid tensor descriptor");
    RCU_REQUIRE(dev, act == RCU_GELU || act == RCU_SILU, "glu: the activation is gelu or silu");
    RCU_REQUIRE(dev, x->dt == dst->dt && dt_is_float(x->dt), "glu: float tensors of one dtype");
    const uint64_t F2 = x->shape[x->rank - 1], rows = t_numel(x) / F2;
    RCU_REQUIRE(dev, F2 % 2 == 0 && t_numel(dst) == rows * (F2 / 2) && F2 <= 0x7fffffffull, "glu: dst must hold half of each row");
    DevGuard g(dev->ordinal);
    switch (x->dt) {
        case RCU_F32: return launch_glu<float>(dev, x->data, dst->data, rows, F2 / 2, act);
        case RCU_F16: return launch_glu<__half>(dev, x->data, dst->data, rows, F2 / 2, act);
        default: return launch_glu<__nv_bfloat16>(dev, x->data, dst->data, rows, F2 / 2, act);
    }
}

rcu_status rcu_rotary_frequencies(uint32_t dims, double base, double factor, double original, double fast, double slow, float* host_freqs,
                                  float* magnitude) {
    if (!host_freqs || !magnitude || dims < 2 || dims % 2 || !(base > 1.0)) return RCU_ERR_INVALID_ARG;
    const bool yarn = factor > 0.0;
    if (yarn && !(original > 0.0 && fast > 0.0 && slow > 0.0)) return RCU_ERR_INVALID_ARG;
    const uint32_t pairs = dims / 2;
    double lo = 0.0, hi = 0.0;
    if (yarn) {
        // index of the pair whose wave turns `t` times over the original length
        auto pair_at = [&](double t) { return dims * std::log(original / (2.0 * M_PI * t)) / (2.0 * std::log(base)); };
        lo = std::fmax(std::floor(pair_at(fast)), 0.0);
        hi = std::fmin(std::ceil(pair_at(slow)), (double)dims - 1.0);
    }
    for (uint32_t i = 0; i < pairs; ++i) {
        double f = std::pow(base, -2.0 * i / dims);
        if (yarn) {
            const double ramp = std::fmin(std::fmax((i - lo) / std::fmax(hi - lo, 0.001), 0.0), 1.0);
            f = f / factor * ramp + f * (1.0 - ramp);
        }
        host_freqs[i] = (float)f;
        host_freqs[pairs + i] = (float)(f - (double)(float)f);
    }
    *magnitude = yarn ? (float)(0.1 * std::log(factor) + 1.0) : 1.0f;
    return RCU_OK;
}

rcu_status rcu_rotary(rcu_device* dev, const rcu_tensor* x, uint32_t first, const rcu_tensor* freqs, float magnitude, uint32_t position, rcu_tensor* dst) {
    if (!dev) return RCU_ERR_INVALID_ARG;
    RCU_REQUIRE(dev, t_valid(x) && t_valid(freqs) && t_valid(dst), "rotary: invalid tensor descriptor");
    RCU_REQUIRE(dev, x->rank == 3 && t_same_shape(x, dst) && x->dt == dst->dt && dt_is_float(x->dt), "rotary: x and dst are float [tokens, heads, dim]");
    RCU_REQUIRE(dev, freqs->dt == RCU_F32 && freqs->rank == 2 && freqs->shape[0] == 2, "rotary: the frequency table is f32 [2, pairs]");
    const uint64_t pairs = freqs->shape[1];
    RCU_REQUIRE(dev, first + 2 * pairs <= x->shape[2] && pairs <= 4096 && x->shape[0] <= 0x7fffffffull, "rotary: the rotated features lie outside the head");
    DevGuard g(dev->ordinal);
#define RCU_ROT(T_)                                                                                                                              \
    rcu_launch(dev, rotary_kernel<T_>, (unsigned)x->shape[0], 128, pairs * sizeof(float2), (const T_*)x->data, (const float*)freqs->data, (T_*)dst->data, \
               (int)x->shape[1], (int)x->shape[2], (int)first, (int)pairs, magnitude, position)
    if (x->dt == RCU_F32) RCU_ROT(float);
    else if (x->dt == RCU_BF16) RCU_ROT(__nv_bfloat16);
    else RCU_ROT(__half);
#undef RCU_ROT
    RCU_LAUNCH_CHECK(dev);
    return RCU_OK;
}

rcu_status rcu_stream_rows(rcu_device* dev, const rcu_tensor* x, int32_t copy_dt, rcu_tensor* dst) {
    if (!dev) return RCU_ERR_INVALID_ARG;
    RCU_REQUIRE(dev, t_valid(x) && t_valid(dst), "stream_rows: invalid tensor descriptor");
    RCU_REQUIRE(dev, x->rank == 2 && dst->rank == 2 && (x->dt == RCU_F32 || x->dt == RCU_BF16) && dst->dt == RCU_F32 && (copy_dt == RCU_F32 || copy_dt == RCU_BF16),
                "stream_rows: f32 or bf16 rows into f32 stream rows");
    const uint64_t W = x->shape[1], pitch = copy_dt == RCU_BF16 ? W + (W + 1) / 2 : W;
    RCU_REQUIRE(dev, dst->shape[0] == x->shape[0] && dst->shape[1] == pitch && x->shape[0] <= 0x7fffffffull && pitch <= 0x7fffffffull,
                "stream_rows: dst rows of %llu words expected", (unsigned long long)pitch);
    DevGuard g(dev->ordinal);
    const unsigned rows = (unsigned)x->shape[0];
    if (x->dt == RCU_F32) rcu_launch(dev, stream_rows_kernel<float>, rows, 256, 0, (const float*)x->data, (float*)dst->data, (int)W, (int)pitch);
    else rcu_launch(dev, stream_rows_kernel<__nv_bfloat16>, rows, 256, 0, (const __nv_bfloat16*)x->data, (float*)dst->data, (int)W, (int)pitch);
    RCU_LAUNCH_CHECK(dev);
    return RCU_OK;
}

rcu_status rcu_post_norm(rcu_device* dev, const rcu_tensor* x, const rcu_tensor* y, const rcu_tensor* scale, const rcu_tensor* shift, float eps,
                         rcu_tensor* dst) {
    if (!dev) return RCU_ERR_INVALID_ARG;
    RCU_REQUIRE(dev, t_valid(x) && t_valid(y) && t_valid(scale) && t_valid(shift) && t_valid(dst), "post_norm: invalid tensor descriptor");
    RCU_REQUIRE(dev, x->dt == RCU_F32 && y->dt == RCU_F32 && scale->dt == RCU_F32 && shift->dt == RCU_F32 && dst->dt == RCU_F32, "post_norm: f32 tensors");
    RCU_REQUIRE(dev, x->rank == 2 && y->rank == 2 && t_same_shape(x, dst) && x->shape[0] == y->shape[0], "post_norm: stream rows and sublayer rows of one count");
    const uint64_t W = y->shape[1], rows = y->shape[0], pitch = x->shape[1];
    RCU_REQUIRE(dev, t_numel(scale) == W && t_numel(shift) == W && (pitch == W || pitch == W + (W + 1) / 2) && rows <= 0x7fffffffull && pitch <= 0x7fffffffull,
                "post_norm: rows of %llu words for a width of %llu", (unsigned long long)pitch, (unsigned long long)W);
    DevGuard g(dev->ordinal);
    const PostNormArgs a{(const float*)x->data, (const float*)y->data, (const float*)scale->data, (const float*)shift->data, (float*)dst->data, (int)W, (int)pitch, eps};
    if (W % 8 == 0 && W <= 8192 &&
        ((reinterpret_cast<uintptr_t>(a.x) | reinterpret_cast<uintptr_t>(a.y) | reinterpret_cast<uintptr_t>(a.scale) | reinterpret_cast<uintptr_t>(a.shift) |
          reinterpret_cast<uintptr_t>(a.out)) & 15) == 0) {
        if (W <= 1024) rcu_launch(dev, post_norm_quad_kernel<1>, (unsigned)rows, 256, 0, a);
        else if (W <= 2048) rcu_launch(dev, post_norm_quad_kernel<2>, (unsigned)rows, 256, 0, a);
        else if (W <= 4096) rcu_launch(dev, post_norm_quad_kernel<4>, (unsigned)rows, 256, 0, a);
        else rcu_launch(dev, post_norm_quad_kernel<8>, (unsigned)rows, 256, 0, a);
    } else {
        rcu_launch(dev, post_norm_kernel, (unsigned)((rows + 7) / 8), 256, 0, a, (long long)rows);
    }
    RCU_LAUNCH_CHECK(dev);
    return RCU_OK;
}

rcu_status rcu_rotary_angles(rcu_device* dev, const rcu_tensor* freqs, float magnitude, uint32_t position, rcu_tensor* dst) {
    if (!dev) return RCU_ERR_INVALID_ARG;
    RCU_REQUIRE(dev, t_valid(freqs) && t_valid(dst) && freqs->dt == RCU_F32 && freqs->rank == 2 && freqs->shape[0] == 2, "rotary_angles: the frequency table is f32 [2, pairs]");
    const uint64_t pairs = freqs->shape[1], n = t_numel(dst) / 2;
    RCU_REQUIRE(dev, dst->dt == RCU_F32 && dst->rank == 2 && dst->shape[1] == 2 * pairs && n / 128 < 0x7fffffffull, "rotary_angles: dst is f32 [tokens, 2 pairs]");
    DevGuard g(dev->ordinal);
    rcu_launch(dev, rotary_angles_kernel, (unsigned)((n + 127) / 128), 128, 0, (const float*)freqs->data, (float2*)dst->data, (int)pairs, magnitude, position, (long long)n);
    RCU_LAUNCH_CHECK(dev);
    return RCU_OK;
}

rcu_status rcu_norm_rotary(rcu_device* dev, const rcu_tensor* x, uint32_t x_col, const rcu_tensor* scale, float eps, const rcu_tensor* angles, rcu_tensor* dst) {
    if (!dev) return RCU_ERR_INVALID_ARG;
    RCU_REQUIRE(dev, t_valid(x) && t_valid(scale) && t_valid(angles) && t_valid(dst), "norm_rotary: invalid tensor descriptor");
    RCU_REQUIRE(dev, (x->dt == RCU_F32 || x->dt == RCU_BF16) && x->dt == dst->dt && scale->dt == RCU_F32 && angles->dt == RCU_F32, "norm_rotary: f32 or bf16 rows");
    RCU_REQUIRE(dev, x->rank == 2 && dst->rank == 3 && angles->rank == 2 && dst->shape[0] == x->shape[0] && angles->shape[0] == x->shape[0] &&
                         t_numel(scale) == dst->shape[2] && angles->shape[1] <= dst->shape[2] && x_col + dst->shape[1] * dst->shape[2] <= x->shape[1],
                "norm_rotary: the heads do not fit the rows");
    RCU_REQUIRE(dev, dst->shape[0] * dst->shape[1] <= 0x7fffffffull && dst->shape[2] <= 65536, "norm_rotary: too many heads");
    DevGuard g(dev->ordinal);
    const lm::HeadNorm a{(const float*)scale->data, (const float*)angles->data, (int)dst->shape[2], (int)(angles->shape[1] / 2), eps};
    const void* xp = (const char*)x->data + (size_t)x_col * dt_esize(x->dt);
    if (x->dt == RCU_F32) launch_norm_rotary<float>(dev, a, xp, (long long)x->shape[1], dst->data, (int)dst->shape[1], (long long)dst->shape[0]);
    else launch_norm_rotary<__nv_bfloat16>(dev, a, xp, (long long)x->shape[1], dst->data, (int)dst->shape[1], (long long)dst->shape[0]);
    RCU_LAUNCH_CHECK(dev);
    return RCU_OK;
}

}  // extern "C"
