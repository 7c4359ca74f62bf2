// Shared by the dense (bfloat16 / fp32) kernels: element types, activations, the epilogue of a linear.
#pragma once
#include <cuda_bf16.h>

#include "../../include/llamatov_b200_dense.h"
#include "lt_common.cuh"

namespace lt {
namespace dn {

typedef __nv_bfloat16 bf16;

template <typename T>
__device__ __forceinline__ float to_f(T v);
template <>
__device__ __forceinline__ float to_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ float to_f<bf16>(bf16 v) { return __bfloat162float(v); }

template <typename T>
__device__ __forceinline__ T from_f(float v);
template <>
__device__ __forceinline__ float from_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16_rn(v); }

// the two bf16 of a 32-bit word as floats (bf16 is the upper half of an fp32)
__device__ __forceinline__ float lo_f(unsigned w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float hi_f(unsigned w) { return __uint_as_float(w & 0xffff0000u); }

// 16 bytes of elements as floats: 8 bf16 or 4 fp32
template <typename T>
struct Vec;
template <>
struct Vec<bf16> {
    static constexpr int N = 8;
    static __device__ __forceinline__ void unpack(const uint4& r, float (&f)[8]) {
        f[0] = lo_f(r.x); f[1] = hi_f(r.x); f[2] = lo_f(r.y); f[3] = hi_f(r.y);
        f[4] = lo_f(r.z); f[5] = hi_f(r.z); f[6] = lo_f(r.w); f[7] = hi_f(r.w);
    }
};
template <>
struct Vec<float> {
    static constexpr int N = 4;
    static __device__ __forceinline__ void unpack(const uint4& r, float (&f)[4]) {
        f[0] = __uint_as_float(r.x); f[1] = __uint_as_float(r.y);
        f[2] = __uint_as_float(r.z); f[3] = __uint_as_float(r.w);
    }
};

// __fdividef: two units in the last place and no slow path (a large e^(-z) gives 0, as it should)
__device__ __forceinline__ float sigmoid_f(float z) { return __fdividef(1.0f, 1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float logsigmoid_f(float z) { return fminf(z, 0.0f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float gelu_tanh_f(float z) {
    return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
// the same where the result is rounded to bf16: fast exponential and division (relative error below 2^-20)
__device__ __forceinline__ float silu_bf16(float v) { return __fdividef(v, 1.0f + __expf(-v)); }
__device__ __forceinline__ float sigmoid_bf16(float v) { return __fdividef(1.0f, 1.0f + __expf(-v)); }
__device__ __forceinline__ float gelu_tanh_bf16(float z) {      // (1 + tanh u) / 2 = 1 / (1 + e^(-2u))
    return __fdividef(z, 1.0f + __expf(-1.5957691216057308f * (z + 0.044715f * z * z * z)));
}
__device__ __forceinline__ float act_f(int act, float v) {
    if (act == LT_DN_ACT_SILU) return v * sigmoid_f(v);
    if (act == LT_DN_ACT_SIGMOID) return sigmoid_f(v);
    if (act == LT_DN_ACT_LOGSIGMOID) return logsigmoid_f(v);
    return v;
}

// Epilogue of one output row n: what does not depend on the token is looked up once.
struct RowEpi {
    int act;
    float scale, bias, ls;
};
__device__ __forceinline__ RowEpi row_epi(const lt_dn_epilogue& e, int n) {
    RowEpi r;
    r.act = LT_DN_ACT_NONE;
    r.scale = 1.0f;
#pragma unroll
    for (int i = LT_DN_MAX_SEG - 1; i >= 0; i--)
        if (i < e.nseg && n < e.seg_end[i]) {
            r.act = e.seg_act[i];
            r.scale = e.seg_scale[i];
        }
    r.bias = e.bias != nullptr ? e.bias[n] : 0.0f;
    r.ls = e.ls != nullptr ? e.ls[n] : 1.0f;
    return r;
}
// act(v + bias) * scale of N values of one row, the branch on the activation outside the loop
template <bool BF16_OUT, int N>
__device__ __forceinline__ void epi_values(const RowEpi& r, float (&v)[N]) {
#pragma unroll
    for (int i = 0; i < N; i++) v[i] += r.bias;
    if (r.act == LT_DN_ACT_SILU) {
#pragma unroll
        for (int i = 0; i < N; i++) v[i] = BF16_OUT ? silu_bf16(v[i]) : v[i] * sigmoid_f(v[i]);
    } else if (r.act == LT_DN_ACT_SIGMOID) {
#pragma unroll
        for (int i = 0; i < N; i++) v[i] = BF16_OUT ? sigmoid_bf16(v[i]) : sigmoid_f(v[i]);
    } else if (r.act == LT_DN_ACT_LOGSIGMOID) {
#pragma unroll
        for (int i = 0; i < N; i++) v[i] = logsigmoid_f(v[i]);
    }
#pragma unroll
    for (int i = 0; i < N; i++) v[i] *= r.scale;
}
__device__ __forceinline__ float epi_value(const RowEpi& r, float v) { return act_f(r.act, v + r.bias) * r.scale; }

// output n of row t; Y has row stride ldy
template <typename T>
__device__ __forceinline__ void epi_store(const lt_dn_epilogue& e, const RowEpi& r, void* Y, long t, int ldy, int n, float v) {
    const long idx = t * ldy + n;
    if (e.kind == LT_DN_RESID) {
        float* y = (float*)Y + idx;
        *y = fmaf(r.ls, v + r.bias, *y);
    } else if (e.tail != nullptr && n >= e.tail_from) {
        e.tail[t * e.ldtail + n - e.tail_from] = epi_value(r, v);
    } else if (e.out_f32) {
        ((float*)Y)[idx] = epi_value(r, v);
    } else {
        ((T*)Y)[idx] = from_f<T>(epi_value(r, v));
    }
}
__device__ __forceinline__ float glu_f(const lt_dn_epilogue& e, float g, float u) {
    if (e.glu_act == LT_DN_GLU_GELU) return gelu_tanh_f(g) * u;
    g = fminf(g, e.glu_limit);
    u = fminf(fmaxf(u, -e.glu_limit), e.glu_limit);
    return g * sigmoid_f(e.glu_alpha * g) * (u + 1.0f);
}
// the same where the result is rounded to bf16, N values (bits of floats) with the branch outside the loop
template <int N>
__device__ __forceinline__ void glu_bf16(const lt_dn_epilogue& e, const int (&g)[N], const int (&u)[N], float (&f)[N]) {
    if (e.glu_act == LT_DN_GLU_GELU) {
#pragma unroll
        for (int i = 0; i < N; i++) f[i] = gelu_tanh_bf16(__int_as_float(g[i])) * __int_as_float(u[i]);
    } else {
        const float lim = e.glu_limit, alpha = e.glu_alpha;
#pragma unroll
        for (int i = 0; i < N; i++) {
            const float a = fminf(__int_as_float(g[i]), lim);
            f[i] = __fdividef(a, 1.0f + __expf(-alpha * a)) * (fminf(fmaxf(__int_as_float(u[i]), -lim), lim) + 1.0f);
        }
    }
}
template <typename T>
__device__ __forceinline__ void glu_store(const lt_dn_epilogue& e, void* Y, long idx, float g, float u) {
    const float v = glu_f(e, g, u);
    if (e.out_f32) ((float*)Y)[idx] = v;
    else ((T*)Y)[idx] = from_f<T>(v);
}

// sum over the lanes of a warp, the result in every lane
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int s = 16; s > 0; s >>= 1) v += __shfl_xor_sync(0xffffffffu, v, s);
    return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int s = 16; s > 0; s >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, s));
    return v;
}

inline int sm_count() {
    static int cache[64] = {0};
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return 148;
    if (cache[dev] == 0) {
        int n = 148;
        cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev);
        cache[dev] = n;
    }
    return cache[dev];
}

// host checks shared by the launchers
inline const char* epi_error(const lt_dn_epilogue* e) {
    if (e == nullptr) return "null epilogue";
    if (e->kind < 0 || e->kind > LT_DN_STORE_GLU) return "unknown epilogue kind";
    if (e->glu_act < 0 || e->glu_act > LT_DN_GLU_CLAMPED) return "unknown gated activation";
    if (e->tail != nullptr && (e->tail_from < 0 || e->ldtail < 1)) return "bad fp32 tail";
    if (e->nseg < 0 || e->nseg > LT_DN_MAX_SEG) return "too many segments";
    return nullptr;
}

}  // namespace dn
}  // namespace lt
