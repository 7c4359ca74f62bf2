// Row operators around the linears: embedding rows, RMS norm over groups (with a gate), concatenation.
#include "lt_dn_common.cuh"

namespace lt {
namespace dn {

template <typename T>
__global__ void __launch_bounds__(256) k_embed(const T* __restrict__ table, int tab_ld, const int* __restrict__ tok, float scale,
                                               const float* __restrict__ nw, float eps, float* __restrict__ x, float* __restrict__ x0,
                                               int E, int ld, int V, int* status) {
    __shared__ float sred[8];
    const int t = blockIdx.x;
    int id = tok[t];
    if (id < 0 || id >= V) {
        if (threadIdx.x == 0) atomicOr(status, LT_STATUS_BAD_TOKEN);
        id = 0;
    }
    const T* row = table + (long)id * tab_ld;
    float inv = 1.0f;
    if (nw != nullptr) {
        float s = 0.0f;
        for (int j = threadIdx.x; j < E; j += blockDim.x) {
            const float v = to_f(row[j]) * scale;
            s = fmaf(v, v, s);
        }
        s = warp_sum(s);
        if ((threadIdx.x & 31) == 0) sred[threadIdx.x >> 5] = s;
        __syncthreads();
        s = 0.0f;
#pragma unroll
        for (int i = 0; i < 8; i++) s += sred[i];
        inv = 1.0f / sqrtf(s / (float)E + eps);
    }
    for (int j = threadIdx.x; j < ld; j += blockDim.x) {
        float v = j < E ? to_f(row[j]) * scale : 0.0f;
        if (nw != nullptr && j < E) v = v * inv * nw[j];
        x[(long)t * ld + j] = v;
        if (x0 != nullptr) x0[(long)t * ld + j] = v;
    }
}

// one CTA per row; a warp per group, or the whole CTA for one group
template <typename T>
__global__ void __launch_bounds__(256) k_norm_rows(const float* __restrict__ x, int ldx, const int* __restrict__ rows,
                                                   const float* __restrict__ w, int w_period, const T* __restrict__ gate, int ldg,
                                                   T* __restrict__ y, int ldy, int N, int group, int count, float eps, int gate_first,
                                                   int seg, int segp) {
    extern __shared__ float sinv[];      // of each group, where groups do not follow the segments
    __shared__ float sred[8];
    const int t = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const float* xr = x + (long)(rows != nullptr ? rows[t] : t) * ldx;
    const T* gr = gate != nullptr ? gate + (long)t * ldg : nullptr;
    T* yr = y + (long)t * ldy;
    if (seg > 0) {
        auto in1 = [&](int j) { return xr[j] * (gate_first ? to_f(gr[j]) : 1.0f); };
        for (int g = warp; g < N / segp * seg / count; g += 8) {
            float s = 0.0f;
            for (int r = g * count + lane; r < (g + 1) * count; r += 32) {
                const float v = in1(r / seg * segp + r % seg);
                s = fmaf(v, v, s);
            }
            s = warp_sum(s);
            if (lane == 0) sinv[g] = 1.0f / sqrtf(s / (float)count + eps);
        }
        __syncthreads();
        for (int j = tid; j < N; j += 256) {
            const int r = j % segp;
            float o = 0.0f;
            if (r < seg) {
                o = in1(j) * sinv[(j / segp * seg + r) / count] * w[j];
                if (gr != nullptr && !gate_first) o *= to_f(gr[j]);
            }
            yr[j] = from_f<T>(o);
        }
        return;
    }
    auto gate4 = [&](int j) {
        if (sizeof(T) == 4) return *(const float4*)(gr + j);
        const uint2 r = *(const uint2*)(gr + j);
        return make_float4(lo_f(r.x), hi_f(r.x), lo_f(r.y), hi_f(r.y));
    };
    auto in4 = [&](int j) {                 // what the norm sees
        float4 v = *(const float4*)(xr + j);
        if (gate_first) {
            const float4 g = gate4(j);
            v.x *= g.x; v.y *= g.y; v.z *= g.z; v.w *= g.w;
        }
        return v;
    };
    auto emit = [&](int j, float inv) {     // four elements
        float4 v = in4(j);
        const float4 ww = *(const float4*)(w + j % w_period);
        v.x = v.x * inv * ww.x; v.y = v.y * inv * ww.y; v.z = v.z * inv * ww.z; v.w = v.w * inv * ww.w;
        if (gr != nullptr && !gate_first) {
            const float4 g = gate4(j);
            v.x *= g.x; v.y *= g.y; v.z *= g.z; v.w *= g.w;
        }
        if (sizeof(T) == 4) {
            *(float4*)(yr + j) = v;
        } else {
            const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
            *(uint2*)(yr + j) = make_uint2(*(const unsigned*)&a, *(const unsigned*)&b);
        }
    };
    auto sq = [&](int j, float s) {
        const float4 v = in4(j);
        return fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, s))));
    };
    if (group == N) {
        float s = 0.0f;
        for (int j = tid * 4; j < N; j += 1024) s = sq(j, s);
        s = warp_sum(s);
        if (lane == 0) sred[warp] = s;
        __syncthreads();
        float tot = 0.0f;
#pragma unroll
        for (int i = 0; i < 8; i++) tot += sred[i];
        const float inv = 1.0f / sqrtf(tot / (float)count + eps);
        for (int j = tid * 4; j < N; j += 1024) emit(j, inv);
    } else {
        for (int g = warp; g < N / group; g += 8) {
            float s = 0.0f;
            for (int j = lane * 4; j < group; j += 128) s = sq(g * group + j, s);
            s = warp_sum(s);
            const float inv = 1.0f / sqrtf(s / (float)count + eps);
            for (int j = lane * 4; j < group; j += 128) emit(g * group + j, inv);
        }
    }
}

template <typename T>
__global__ void __launch_bounds__(256) k_concat_rows(const float* __restrict__ x, int ldx, int n1, const float* __restrict__ x2,
                                                     int ldx2, int n2, T* __restrict__ y, int ldy) {
    const long t = blockIdx.x;
    for (int j = threadIdx.x; j < n1 + n2; j += blockDim.x)
        y[t * ldy + j] = from_f<T>(j < n1 ? x[t * ldx + j] : x2[t * ldx2 + j - n1]);
}

}  // namespace dn
}  // namespace lt

using namespace lt;
using namespace lt::dn;

extern "C" int lt_dn_embed(const void* table, int f32, int tab_ld, const int* tok, float scale, const float* norm_w, float eps, float* x,
                           float* x0, int E, int ld, int V, int T, void* stream) {
    LT_REQUIRE(table && tok && x, "lt_dn_embed: null pointer");
    LT_REQUIRE(E > 0 && ld >= E && tab_ld >= E && V > 0 && T > 0, "lt_dn_embed: E=%d ld=%d tab_ld=%d V=%d T=%d", E, ld, tab_ld, V, T);
    int* st = device_status_ptr();
    LT_REQUIRE(st != nullptr, "lt_dn_embed: status word unavailable");
    if (f32) k_embed<float><<<T, 256, 0, (cudaStream_t)stream>>>((const float*)table, tab_ld, tok, scale, norm_w, eps, x, x0, E, ld, V, st);
    else k_embed<bf16><<<T, 256, 0, (cudaStream_t)stream>>>((const bf16*)table, tab_ld, tok, scale, norm_w, eps, x, x0, E, ld, V, st);
    return check_launch("lt_dn_embed");
}

extern "C" int lt_dn_norm_rows(const float* x, int ldx, const int* rows, const float* w, int w_period, const void* gate, int ldg,
                               void* y, int ldy, int f32, int T, int N, int group, int count, float eps, int gate_first, int seg, int segp,
                               void* stream) {
    LT_REQUIRE(x && w && y && (!gate_first || gate), "lt_dn_norm_rows: null pointer");
    LT_REQUIRE(T > 0 && N > 0 && N % 4 == 0 && count > 0 && w_period > 0 && w_period % 4 == 0,
               "lt_dn_norm_rows: T=%d N=%d count=%d w_period=%d", T, N, count, w_period);
    size_t smem = 0;
    if (seg > 0) {
        LT_REQUIRE(segp >= seg && N % segp == 0 && (N / segp * seg) % count == 0 && w_period >= N,
                   "lt_dn_norm_rows: segments of %d in %d, groups of %d", seg, segp, count);
        smem = (size_t)(N / segp * seg / count) * 4;
        LT_REQUIRE(smem <= 40 * 1024, "lt_dn_norm_rows: too many groups of %d", count);
    } else {
        LT_REQUIRE(group > 0 && group % 4 == 0 && N % group == 0, "lt_dn_norm_rows: group=%d of N=%d", group, N);
    }
    LT_REQUIRE(ldx % 4 == 0 && ldx >= N && ldy % 4 == 0 && ldy >= N && ldg % 4 == 0 && aligned16(x) && aligned16(w) && aligned16(y) &&
                   aligned16(gate),
               "lt_dn_norm_rows: ldx=%d ldy=%d ldg=%d N=%d", ldx, ldy, ldg, N);
    cudaStream_t s = (cudaStream_t)stream;
    if (f32) k_norm_rows<float><<<T, 256, smem, s>>>(x, ldx, rows, w, w_period, (const float*)gate, ldg, (float*)y, ldy, N, group, count, eps, gate_first, seg, segp);
    else k_norm_rows<bf16><<<T, 256, smem, s>>>(x, ldx, rows, w, w_period, (const bf16*)gate, ldg, (bf16*)y, ldy, N, group, count, eps, gate_first, seg, segp);
    return check_launch("lt_dn_norm_rows");
}

extern "C" int lt_dn_concat_rows(const float* x, int ldx, int n1, const float* x2, int ldx2, int n2, void* y, int ldy, int f32, int T,
                                 void* stream) {
    LT_REQUIRE(x && x2 && y && T > 0 && n1 > 0 && n2 >= 0 && ldy >= n1 + n2, "lt_dn_concat_rows: T=%d n1=%d n2=%d ldy=%d", T, n1, n2, ldy);
    cudaStream_t s = (cudaStream_t)stream;
    if (f32) k_concat_rows<float><<<T, 256, 0, s>>>(x, ldx, n1, x2, ldx2, n2, (float*)y, ldy);
    else k_concat_rows<bf16><<<T, 256, 0, s>>>(x, ldx, n1, x2, ldx2, n2, (bf16*)y, ldy);
    return check_launch("lt_dn_concat_rows");
}
