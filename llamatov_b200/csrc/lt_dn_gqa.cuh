// Host check of the description of a grouped-query attention layer, and the rotation both of its kernels use.
#pragma once
#include <limits.h>

#include "lt_dn_common.cuh"

namespace lt {
namespace dn {

// cos and sin of pos * (hi + lo): the rounding of the product and lo are a small angle added in first order
__device__ __forceinline__ void rotation(int pos, float2 f, float& c, float& s) {
    const float p = (float)pos, a = p * f.x, e = fmaf(p, f.x, -a) + p * f.y;
    float s0, c0;
    sincosf(a, &s0, &c0);
    c = fmaf(-e, s0, c0);
    s = fmaf(e, c0, s0);
}

inline const char* gqa_error(const lt_dn_gqa* A) {
    if (A == nullptr) return "null description";
    if (A->H <= 0 || A->G <= 0 || A->H % A->G || A->dp <= 0 || A->dvp <= 0) return "heads and head sizes";
    if (A->dp % 8 || A->dvp % 8) return "padded sizes must be multiples of 8";
    if (A->rot < 0 || A->rot % 2 || A->rot > A->dp) return "rotated dimensions must be even and fit the head";
    if (A->qcount <= 0 || A->kcount <= 0 || A->cap <= 0) return "norm counts and cache rows must be positive";
    if (!(A->softcap >= 0.0f)) return "negative softcap";
    if (A->qnorm == nullptr || A->knorm == nullptr || (A->rot > 0 && A->freq == nullptr)) return "null constants";
    return nullptr;
}

}  // namespace dn
}  // namespace lt
