// Grouped-query attention over a cache of plain key and value rows: queries and keys are RMS-normed over their whole
// projection and rotated, values may be mixed with those of an earlier layer, scores may be capped, heads may be gated.
//
// k_gqa_rows prepares the rows of a portion (lt_dn_gqa_attn in lt_dn_attn.cu follows).  k_gqa_step is a whole token: every CTA
// takes one range of positions for up to SH query heads of one key head; the CTA whose range ends at the new position makes
// the new key and value itself and appends them; the CTA that finishes last of its heads combines the ranges.
#include "lt_dn_gqa.cuh"
#include "lt_dn_mma.cuh"

namespace lt {
namespace dn {

// (1 - m) v + m v0
__device__ __forceinline__ float mix_value(float v, float v0, float m) { return fmaf(m, v0, (1.0f - m) * v); }

// Sum of squares of n elements (a multiple of 8) of this thread's share
template <typename T>
__device__ __forceinline__ float square_sum(const T* __restrict__ x, int n, int tid, int nthr) {
    constexpr int N = Vec<T>::N;
    float s = 0.0f;
    for (int j = tid * N; j < n; j += nthr * N) {
        float f[N];
        Vec<T>::unpack(*(const uint4*)(x + j), f);
#pragma unroll
        for (int i = 0; i < N; i++) s = fmaf(f[i], f[i], s);
    }
    return s;
}
template <typename T>
__device__ __forceinline__ void store_vec(T* p, const float (&f)[Vec<T>::N]);
template <>
__device__ __forceinline__ void store_vec<float>(float* p, const float (&f)[4]) { *(float4*)p = make_float4(f[0], f[1], f[2], f[3]); }
template <>
__device__ __forceinline__ void store_vec<bf16>(bf16* p, const float (&f)[8]) {
    unsigned u[4];
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const __nv_bfloat162 h = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
        u[i] = *(const unsigned*)&h;
    }
    *(uint4*)p = make_uint4(u[0], u[1], u[2], u[3]);
}

// ---------------------------------------------------------------------------- rows of a portion

template <typename T>
__global__ void __launch_bounds__(256) k_gqa_rows(T* __restrict__ y, int ld, T* __restrict__ kc, T* __restrict__ vc,
                                                  T* __restrict__ vfirst, int vstore, int pos0, const __grid_constant__ lt_dn_gqa A) {
    constexpr int N = Vec<T>::N;
    extern __shared__ __align__(16) float sm[];     // cos, sin
    __shared__ float sred[2][8];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int t = blockIdx.x, pos = pos0 + t, half = A.rot >> 1;
    const int nq = A.H * A.dp, nk = A.G * A.dp, nv = A.G * A.dvp;
    float* sc = sm;
    float* ss = sm + half;
    for (int i = tid; i < half; i += 256) rotation(pos, ((const float2*)A.freq)[i], sc[i], ss[i]);
    T* row = y + (long)t * ld;
    const float a = warp_sum(square_sum(row, nq, tid, 256)), b = warp_sum(square_sum(row + nq, nk, tid, 256));
    if (lane == 0) {
        sred[0][warp] = a;
        sred[1][warp] = b;
    }
    __syncthreads();
    float qs = 0.0f, ks = 0.0f;
#pragma unroll
    for (int i = 0; i < 8; i++) {
        qs += sred[0][i];
        ks += sred[1][i];
    }
    const float qi = 1.0f / sqrtf(qs / (float)A.qcount + A.eps), ki = 1.0f / sqrtf(ks / (float)A.kcount + A.eps);
    T* krow = kc + (long)pos * nk;
    if (half % N == 0) {
        // units of N elements: pairs of units that rotate, then units that only get the norm
        const int hu = half / N, per = hu + (A.dp - A.rot) / N;
        for (int e = tid; e < (A.H + A.G) * per; e += 256) {
            const int h = e / per, u = e - h * per;
            const bool key = h >= A.H;
            const T* src = row + (long)h * A.dp;
            T* dst = key ? krow + (long)(h - A.H) * A.dp : row + (long)h * A.dp;
            const float* w = key ? A.knorm + (long)(h - A.H) * A.dp : A.qnorm + (long)h * A.dp;
            const float inv = key ? ki : qi;
            if (u < hu) {
                const int j = u * N;
                float f[N], g[N], o[N], p[N];
                Vec<T>::unpack(*(const uint4*)(src + j), f);
                Vec<T>::unpack(*(const uint4*)(src + j + half), g);
#pragma unroll
                for (int i = 0; i < N; i++) {
                    const float x = f[i] * inv * w[j + i], z = g[i] * inv * w[j + half + i];
                    o[i] = x * sc[j + i] - z * ss[j + i];
                    p[i] = z * sc[j + i] + x * ss[j + i];
                }
                store_vec<T>(dst + j, o);
                store_vec<T>(dst + j + half, p);
            } else {
                const int j = A.rot + (u - hu) * N;
                float f[N];
                Vec<T>::unpack(*(const uint4*)(src + j), f);
#pragma unroll
                for (int i = 0; i < N; i++) f[i] = f[i] * inv * w[j + i];
                store_vec<T>(dst + j, f);
            }
        }
    } else {
        const int per = half + A.dp - A.rot;
        for (int e = tid; e < (A.H + A.G) * per; e += 256) {
            const int h = e / per, j = e - h * per;
            const bool key = h >= A.H;
            const T* src = row + (long)h * A.dp;
            T* dst = key ? krow + (long)(h - A.H) * A.dp : row + (long)h * A.dp;
            const float* w = key ? A.knorm + (long)(h - A.H) * A.dp : A.qnorm + (long)h * A.dp;
            const float inv = key ? ki : qi;
            if (j < half) {
                const float x = to_f(src[j]) * inv * w[j], z = to_f(src[j + half]) * inv * w[j + half];
                dst[j] = from_f<T>(x * sc[j] - z * ss[j]);
                dst[j + half] = from_f<T>(z * sc[j] + x * ss[j]);
            } else {
                dst[j + half] = from_f<T>(to_f(src[j + half]) * inv * w[j + half]);
            }
        }
    }
    const T* v = row + nq + nk;
    T* vrow = vc + (long)pos * nv;
    T* vf = vfirst != nullptr ? vfirst + (long)t * nv : nullptr;
    for (int j = tid * N; j < nv; j += 256 * N) {
        uint4 x = *(const uint4*)(v + j);
        if (vf != nullptr && vstore) *(uint4*)(vf + j) = x;
        if (vf != nullptr && !vstore) {
            float f[N], g[N];
            Vec<T>::unpack(x, f);
            Vec<T>::unpack(*(const uint4*)(vf + j), g);
#pragma unroll
            for (int i = 0; i < N; i++) f[i] = mix_value(f[i], g[i], A.vmix);
            store_vec<T>(vrow + j, f);
        } else {
            *(uint4*)(vrow + j) = x;
        }
    }
}

// ---------------------------------------------------------------------------- one token

constexpr int SH = 8;          // query heads of a CTA
constexpr int GT = 128;        // threads
constexpr int MIN_ROWS = 16;   // positions of a range, at least

struct GqaStepP {
    const void* y;
    void *kc, *vc, *vfirst;
    const float* gate;
    void* out;
    int *len, *tickets, *status;
    float *pm, *pl, *pu;       // per range and head: maximum, sum, weighted sum of values
    int splits, nb, vstore, sr;
    lt_dn_gqa A;
};

// RD: value columns per thread / 2 (a thread owns columns 2 c and 2 c + 1, c = its column index + 128 i)
template <typename T, int RD>
__global__ void __launch_bounds__(GT) k_gqa_step(const __grid_constant__ GqaStepP P) {
    constexpr int N = Vec<T>::N;
    extern __shared__ __align__(16) unsigned char smem[];
    const lt_dn_gqa& A = P.A;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int half = A.rot >> 1, per = A.H / A.G, SR = P.sr;
    const int g = blockIdx.y / P.nb, hb = blockIdx.y - g * P.nb, h0 = g * per + hb * SH, nh = min(SH, per - hb * SH);
    const int nq = A.H * A.dp, nk = A.G * A.dp, nv = A.G * A.dvp;
    const int ku = (A.dp / N) | 1, vu = (A.dvp / N) | 1;       // 16-byte units of a staged row: an odd number
    T* sKV = (T*)smem;                                         // two stages of SR key rows, then SR value rows
    const int stage = SR * (ku + vu) * N;
    float* sQ = (float*)(sKV + 2 * stage);                     // [SH][dp]
    float* sP = sQ + SH * A.dp;                                // [SR][SH]
    float* sc = sP + SR * SH;                                  // cos, sin
    float* ss = sc + half;
    T* sNew = (T*)(sc + ((A.rot + 3) & ~3));                   // the new key and value of this key head
    __shared__ float sF[SH], sred[2][GT / 32], sL[SH];
    __shared__ int sflag;

    int pos = *P.len;
    if (pos < 0 || pos >= A.cap) {
        if (tid == 0) atomicOr(P.status, LT_STATUS_KV_OVERFLOW);
        pos = pos < 0 ? 0 : A.cap - 1;
    }
    const int n = pos + 1;
    const int span = max((n + P.splits - 1) / P.splits, MIN_ROWS), active = (n + span - 1) / span;
    const int lo = blockIdx.x * span, hi = min(n, lo + span);
    if ((int)blockIdx.x < active) {
        const bool own = hi == n;
        const T* kbase = (const T*)P.kc + (long)g * A.dp;
        const T* vbase = (const T*)P.vc + (long)g * A.dvp;
        auto fetch = [&](int p0, int b) {
            T* k = sKV + b * stage;
            T* v = k + SR * ku * N;
            const int cu = A.dp / N, cv = A.dvp / N, nr = min(SR, min(hi, pos) - p0);     // the new row is not in memory yet
            for (int e = tid; e < nr * cu; e += GT) {
                const int r = e / cu, c = e - r * cu;
                cp16(k + (r * ku + c) * N, kbase + (long)(p0 + r) * nk + c * N, true);
            }
            for (int e = tid; e < nr * cv; e += GT) {
                const int r = e / cv, c = e - r * cv;
                cp16(v + (r * vu + c) * N, vbase + (long)(p0 + r) * nv + c * N, true);
            }
            asm volatile("cp.async.commit_group;" ::: "memory");
        };
        fetch(lo, 0);

        // ---- queries of this CTA; the new key and value where the range ends at the new position
        const T* row = (const T*)P.y;
        for (int e = tid * N; e < nh * A.dp; e += GT * N) {      // query times norm weight, before the norm is known
            float f[N];
            Vec<T>::unpack(*(const uint4*)(row + (long)h0 * A.dp + e), f);
            const float4* w = (const float4*)(A.qnorm + (long)h0 * A.dp + e);
#pragma unroll
            for (int i = 0; i < N / 4; i++) {
                const float4 x = w[i];
                *(float4*)(sQ + e + 4 * i) = make_float4(f[4 * i] * x.x, f[4 * i + 1] * x.y, f[4 * i + 2] * x.z, f[4 * i + 3] * x.w);
            }
        }
        for (int i = tid; i < half; i += GT) rotation(pos, ((const float2*)A.freq)[i], sc[i], ss[i]);
        const float a = warp_sum(square_sum(row, nq, tid, GT)), b = own ? warp_sum(square_sum(row + nq, nk, tid, GT)) : 0.0f;
        if (lane == 0) {
            sred[0][warp] = a;
            sred[1][warp] = b;
        }
        __syncthreads();
        float qs = 0.0f, ks = 0.0f;
#pragma unroll
        for (int i = 0; i < GT / 32; i++) {
            qs += sred[0][i];
            ks += sred[1][i];
        }
        const float qi = 1.0f / sqrtf(qs / (float)A.qcount + A.eps), ki = 1.0f / sqrtf(ks / (float)A.kcount + A.eps);
        for (int e = tid; e < nh * (A.dp - half); e += GT) {     // half pairs that rotate, then the rest of the head
            const int h = e / (A.dp - half), i = e - h * (A.dp - half);
            float* x = sQ + h * A.dp + i;
            const float u = x[i < half ? 0 : half] * qi;
            if (i < half) {
                const float z = x[half] * qi;
                x[0] = to_f(from_f<T>(u * sc[i] - z * ss[i]));
                x[half] = to_f(from_f<T>(z * sc[i] + u * ss[i]));
            } else {
                x[half] = to_f(from_f<T>(u));
            }
        }
        // element j of the normed, rotated key
        auto turned = [&](const T* x, const float* w, float inv, int j) {
            const float u = to_f(x[j]) * inv * w[j];
            if (j >= A.rot) return u;
            const int i = j < half ? j : j - half, o = j < half ? j + half : j - half;
            const float z = to_f(x[o]) * inv * w[o];
            return j < half ? u * sc[i] - z * ss[i] : u * sc[i] + z * ss[i];
        };
        if (own) {
            T* kr = (T*)P.kc + (long)pos * nk + (long)g * A.dp;
            T* vr = (T*)P.vc + (long)pos * nv + (long)g * A.dvp;
            for (int j = tid; j < A.dp; j += GT) {
                const T k = from_f<T>(turned(row + nq + (long)g * A.dp, A.knorm + (long)g * A.dp, ki, j));
                sNew[j] = k;
                if (hb == 0) kr[j] = k;
            }
            T* vf = P.vfirst != nullptr ? (T*)P.vfirst + (long)g * A.dvp : nullptr;
            for (int j = tid; j < A.dvp; j += GT) {
                T v = row[nq + nk + (long)g * A.dvp + j];
                if (vf != nullptr && P.vstore && hb == 0) vf[j] = v;
                if (vf != nullptr && !P.vstore) v = from_f<T>(mix_value(to_f(v), to_f(vf[j]), A.vmix));
                sNew[A.dp + j] = v;
                if (hb == 0) vr[j] = v;
            }
        }

        // ---- the range, SR positions at a time
        const int ncp = A.dvp >> 1;                   // column pairs
        int cw = 1;                                   // threads of a row group: column pairs, rounded up to a power of two
        while (cw < ncp && cw < GT) cw <<= 1;
        const int rg = tid / cw, nrg = GT / cw, cp = tid & (cw - 1);
        float acc[RD][SH][2];
#pragma unroll
        for (int i = 0; i < RD; i++)
#pragma unroll
            for (int h = 0; h < SH; h++) acc[i][h][0] = acc[i][h][1] = 0.0f;
        float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};      // of heads warp and warp + 4
        int buf = 0;
        for (int p0 = lo; p0 < hi; p0 += SR, buf ^= 1) {
            const int nr = min(SR, hi - p0);
            T* k = sKV + buf * stage;
            T* v = k + SR * ku * N;
            if (p0 + SR < hi) {
                fetch(p0 + SR, buf ^ 1);
                asm volatile("cp.async.wait_group 1;" ::: "memory");
            } else {
                asm volatile("cp.async.wait_group 0;" ::: "memory");
            }
            __syncthreads();
            if (own && p0 + nr == n) {
                const int r = nr - 1;
                for (int j = tid; j < A.dp; j += GT) k[r * ku * N + j] = sNew[j];
                for (int j = tid; j < A.dvp; j += GT) v[r * vu * N + j] = sNew[A.dp + j];
                __syncthreads();
            }
            // scores: a lane has a row, a warp two heads
            const int npair = (nh + 1) >> 1, nblk = (nr + 31) >> 5;
            for (int it = warp; it < npair * nblk; it += GT / 32) {
                const int hp = it % npair, r = (it / npair) * 32 + lane;
                const float* q0 = sQ + 2 * hp * A.dp;
                const float* q1 = q0 + A.dp;
                const T* kr = k + min(r, nr - 1) * ku * N;
                float s0 = 0.0f, s1 = 0.0f;
                for (int c = 0; c < A.dp; c += N) {
                    float f[N];
                    Vec<T>::unpack(*(const uint4*)(kr + c), f);
#pragma unroll
                    for (int i = 0; i < N; i += 4) {
                        const float4 x = *(const float4*)(q0 + c + i), z = *(const float4*)(q1 + c + i);
                        s0 = fmaf(f[i], x.x, fmaf(f[i + 1], x.y, fmaf(f[i + 2], x.z, fmaf(f[i + 3], x.w, s0))));
                        s1 = fmaf(f[i], z.x, fmaf(f[i + 1], z.y, fmaf(f[i + 2], z.z, fmaf(f[i + 3], z.w, s1))));
                    }
                }
                s0 *= A.scale;
                s1 *= A.scale;
                if (A.softcap > 0.0f) {
                    s0 = A.softcap * tanhf(s0 / A.softcap);
                    s1 = A.softcap * tanhf(s1 / A.softcap);
                }
                if (r < nr) *(float2*)(sP + r * SH + 2 * hp) = make_float2(s0, s1);
            }
            __syncthreads();
            // softmax over the rows so far: a warp has two heads
#pragma unroll
            for (int i = 0; i < 2; i++) {
                const int h = warp + i * (GT / 32);
                if (h >= nh) continue;
                float mx = m[i];
                for (int r = lane; r < nr; r += 32) mx = fmaxf(mx, sP[r * SH + h]);
                mx = warp_max(mx);
                const float f = expf(m[i] - mx);
                float sum = 0.0f;
                for (int r = lane; r < nr; r += 32) {
                    const float p = expf(sP[r * SH + h] - mx);
                    sP[r * SH + h] = p;
                    sum += p;
                }
                m[i] = mx;
                l[i] = l[i] * f + warp_sum(sum);
                if (lane == 0) sF[h] = f;
            }
            __syncthreads();
#pragma unroll
            for (int h = 0; h < SH; h++) {
                if (h >= nh) break;
                const float f = sF[h];
#pragma unroll
                for (int i = 0; i < RD; i++) {
                    acc[i][h][0] *= f;
                    acc[i][h][1] *= f;
                }
            }
            for (int r = rg; r < nr; r += nrg) {
                float p[SH];
#pragma unroll
                for (int h = 0; h < SH; h += 4) {
                    if (h >= nh) break;
                    const float4 x = *(const float4*)(sP + r * SH + h);
                    p[h] = x.x; p[h + 1] = x.y; p[h + 2] = x.z; p[h + 3] = x.w;
                }
#pragma unroll
                for (int i = 0; i < RD; i++) {
                    const int c = cp + GT * i;
                    if (c >= ncp) continue;
                    const float x = to_f(v[r * vu * N + 2 * c]), z = to_f(v[r * vu * N + 2 * c + 1]);
#pragma unroll
                    for (int h = 0; h < SH; h++) {
                        if (h >= nh) break;
                        acc[i][h][0] = fmaf(p[h], x, acc[i][h][0]);
                        acc[i][h][1] = fmaf(p[h], z, acc[i][h][1]);
                    }
                }
            }
            __syncthreads();
        }

        // ---- partial results: row groups are summed in shared memory
        const long pb = (long)blockIdx.x * A.H + h0;
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const int h = warp + i * (GT / 32);
            if (h < nh && lane == 0) {
                P.pm[pb + h] = m[i];
                P.pl[pb + h] = l[i];
            }
        }
        float* sA = (float*)smem;                     // [nrg][SH][2 ncp]
        if (nrg > 1) {
#pragma unroll
            for (int h = 0; h < SH; h++)
                if (h < nh && cp < ncp) *(float2*)(sA + (rg * SH + h) * A.dvp + 2 * cp) = make_float2(acc[0][h][0], acc[0][h][1]);
            __syncthreads();
            for (int e = tid; e < nh * A.dvp; e += GT) {
                float s = 0.0f;
                for (int i = 0; i < nrg; i++) s += sA[i * SH * A.dvp + e];
                P.pu[pb * A.dvp + e] = s;
            }
        } else {
#pragma unroll
            for (int i = 0; i < RD; i++)
#pragma unroll
                for (int h = 0; h < SH; h++)
                    if (h < nh && cp + GT * i < ncp)
                        *(float2*)(P.pu + (pb + h) * A.dvp + 2 * (cp + GT * i)) = make_float2(acc[i][h][0], acc[i][h][1]);
        }
    }

    // ---- the last CTA of these heads combines
    __threadfence();
    __syncthreads();
    if (tid == 0) sflag = atomicAdd(P.tickets + blockIdx.y, 1) == (int)gridDim.x - 1;
    __syncthreads();
    if (!sflag) return;
    __threadfence();
    float* sw = (float*)smem;                         // [SH][active]
    for (int h = warp; h < nh; h += GT / 32) {
        float mx = -INFINITY;
        for (int s = lane; s < active; s += 32) mx = fmaxf(mx, __ldcg(P.pm + (long)s * A.H + h0 + h));
        mx = warp_max(mx);
        float sum = 0.0f;
        for (int s = lane; s < active; s += 32) {
            const float w = expf(__ldcg(P.pm + (long)s * A.H + h0 + h) - mx);
            sw[h * active + s] = w;
            sum = fmaf(w, __ldcg(P.pl + (long)s * A.H + h0 + h), sum);
        }
        sum = warp_sum(sum);
        if (lane == 0) sL[h] = (P.gate != nullptr ? P.gate[h0 + h] : 1.0f) / sum;
    }
    __syncthreads();
    const int nq4 = A.dvp >> 2;
    for (int e = tid; e < nh * nq4; e += GT) {
        const int h = e / nq4, c = (e - h * nq4) * 4;
        const float* u = P.pu + (long)(h0 + h) * A.dvp + c;
        float4 o = make_float4(0, 0, 0, 0);
#pragma unroll 16
        for (int s = 0; s < active; s++) {
            const float4 x = __ldcg((const float4*)(u + (long)s * A.H * A.dvp));
            const float w = sw[h * active + s];
            o.x = fmaf(w, x.x, o.x); o.y = fmaf(w, x.y, o.y); o.z = fmaf(w, x.z, o.z); o.w = fmaf(w, x.w, o.w);
        }
        T* out = (T*)P.out + (long)(h0 + h) * A.dvp + c;
        const float f = sL[h];
        out[0] = from_f<T>(o.x * f); out[1] = from_f<T>(o.y * f); out[2] = from_f<T>(o.z * f); out[3] = from_f<T>(o.w * f);
    }
    if (tid == 0) {
        P.tickets[blockIdx.y] = 0;
        if (atomicAdd(P.tickets + gridDim.y, 1) == (int)gridDim.y - 1) {     // every CTA has read the position
            P.tickets[gridDim.y] = 0;
            *P.len = pos + 1;
        }
    }
}

template <typename T>
static int launch_step(const GqaStepP& P, size_t smem, cudaStream_t s) {
    static PerDeviceOnce once;
    if (once.first()) {
        LT_CUDA(cudaFuncSetAttribute(k_gqa_step<T, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
        LT_CUDA(cudaFuncSetAttribute(k_gqa_step<T, 2>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
    }
    const dim3 grid(P.splits, P.A.G * P.nb);
    if (P.A.dvp <= 2 * GT) k_gqa_step<T, 1><<<grid, GT, smem, s>>>(P);
    else k_gqa_step<T, 2><<<grid, GT, smem, s>>>(P);
    return check_launch("lt_dn_gqa_step");
}

}  // namespace dn
}  // namespace lt

using namespace lt;
using namespace lt::dn;

extern "C" int lt_dn_gqa_rows(void* y, int ld, void* kc, void* vc, void* vfirst, int vmix_store, int f32, int T, int pos0,
                              const lt_dn_gqa* h_a, void* stream) {
    const char* bad = gqa_error(h_a);
    LT_REQUIRE(bad == nullptr, "lt_dn_gqa_rows: %s", bad);
    LT_REQUIRE(y && kc && vc, "lt_dn_gqa_rows: null pointer");
    LT_REQUIRE(T > 0 && pos0 >= 0 && pos0 + T <= h_a->cap, "lt_dn_gqa_rows: positions %d .. %d of a cache of %d", pos0, pos0 + T, h_a->cap);
    LT_REQUIRE(ld % 8 == 0 && ld >= (h_a->H + h_a->G) * h_a->dp + h_a->G * h_a->dvp && aligned16(y) && aligned16(kc) && aligned16(vc) &&
                   aligned16(vfirst),
               "lt_dn_gqa_rows: ld=%d, or alignment", ld);
    const size_t smem = (size_t)(h_a->rot + 2) * 4;
    cudaStream_t s = (cudaStream_t)stream;
    if (f32) k_gqa_rows<float><<<T, 256, smem, s>>>((float*)y, ld, (float*)kc, (float*)vc, (float*)vfirst, vmix_store, pos0, *h_a);
    else k_gqa_rows<bf16><<<T, 256, smem, s>>>((bf16*)y, ld, (bf16*)kc, (bf16*)vc, (bf16*)vfirst, vmix_store, pos0, *h_a);
    return check_launch("lt_dn_gqa_rows");
}

extern "C" long lt_dn_gqa_step_ws(int H, int dvp, int splits) { return (long)splits * H * (dvp + 2) + 16; }
extern "C" int lt_dn_gqa_step_tickets(int H, int G) { return G * ((H / G + SH - 1) / SH) + 1; }

extern "C" int lt_dn_gqa_step(const void* y, void* kc, void* vc, void* vfirst, int vmix_store, const float* gate, void* out, int f32,
                              int* len, const lt_dn_gqa* h_a, int splits, float* ws, int* tickets, void* stream) {
    const char* bad = gqa_error(h_a);
    LT_REQUIRE(bad == nullptr, "lt_dn_gqa_step: %s", bad);
    LT_REQUIRE(y && kc && vc && out && len && ws && tickets, "lt_dn_gqa_step: null pointer");
    LT_REQUIRE(splits > 0 && splits <= 1024, "lt_dn_gqa_step: splits=%d", splits);
    LT_REQUIRE(h_a->dvp <= 4 * GT, "lt_dn_gqa_step: value size %d of a head is above %d", h_a->dvp, 4 * GT);
    LT_REQUIRE(aligned16(y) && aligned16(kc) && aligned16(vc) && aligned16(ws) && aligned16(h_a->qnorm), "lt_dn_gqa_step: pointers must be 16-byte aligned");
    GqaStepP P = {};
    P.y = y; P.kc = kc; P.vc = vc; P.vfirst = vfirst; P.gate = gate; P.out = out; P.len = len; P.tickets = tickets;
    P.status = device_status_ptr();
    LT_REQUIRE(P.status != nullptr, "lt_dn_gqa_step: status word unavailable");
    P.splits = splits; P.vstore = vmix_store; P.A = *h_a;
    P.nb = (h_a->H / h_a->G + SH - 1) / SH;
    P.pu = ws;
    P.pm = P.pu + (long)splits * h_a->H * h_a->dvp;
    P.pl = P.pm + (long)splits * h_a->H;
    const int N = f32 ? 4 : 8, e = f32 ? 4 : 2;
    const size_t unit = (size_t)((h_a->dp / N) | 1) + ((h_a->dvp / N) | 1);
    const size_t fixed = (size_t)(SH * h_a->dp + ((h_a->rot + 3) & ~3)) * 4 + (size_t)(h_a->dp + h_a->dvp) * e + 16;
    const size_t tail = (size_t)SH * splits * 4, rows = (size_t)SH * 2 * GT * 4;       // the stages are reused for these
    auto bytes = [&](int sr) {
        size_t st = 2 * sr * unit * 16;
        const size_t all = st + (size_t)sr * SH * 4 + fixed;
        return all > tail ? (all > rows ? all : rows) : (tail > rows ? tail : rows);
    };
    P.sr = bytes(64) <= 100 * 1024 ? 64 : bytes(32) <= 220 * 1024 ? 32 : 16;
    const size_t smem = bytes(P.sr);
    LT_REQUIRE(smem <= 220 * 1024, "lt_dn_gqa_step: head sizes %d, %d need %zu bytes of shared memory", h_a->dp, h_a->dvp, smem);
    if (f32) return launch_step<float>(P, smem, (cudaStream_t)stream);
    return launch_step<bf16>(P, smem, (cudaStream_t)stream);
}
