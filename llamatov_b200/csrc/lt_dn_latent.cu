// Windowed attention over a latent cache: per position one row [c, kr], c the normed latent that keys and values of
// every head are projections of, kr the rotated key part the heads share.
//
// Prompt portions (lt_dn_latent_rows, then the key/value expansion by lt_dn_linear, then lt_dn_window_attn): keys and
// values of the portion and of the window before it are expanded per head.
// One token (lt_dn_latent_step, three launches): nothing is expanded.  The query is taken through W_uk^T, scores and
// the weighted sum are over the latent rows (all heads read the same rows), and the value projection is applied to the
// sum.
#include "lt_dn_latent.cuh"
#include "lt_dn_mma.cuh"

namespace lt {
namespace dn {

// ---------------------------------------------------------------------------- rows of a portion

template <typename T>
__global__ void __launch_bounds__(256) k_latent_rows(T* __restrict__ y, int ld, T* __restrict__ ring, T* __restrict__ keys, int np,
                                                     int pos0, int nrow, const __grid_constant__ lt_dn_latent L) {
    extern __shared__ __align__(16) float sm[];     // cos, sin
    __shared__ float sred[8];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int half = L.rot >> 1, wr = L.rp + L.rtp;
    if ((int)blockIdx.x >= nrow) {     // an earlier row of the window
        const int i = blockIdx.x - nrow;
        const T* src = ring + (long)((pos0 - np + i) % L.cap) * wr;
        for (int j = tid; j < wr; j += 256) keys[(long)i * wr + j] = src[j];
        return;
    }
    const int t = blockIdx.x, pos = pos0 + t;
    float* sc = sm;
    float* ss = sm + half;
    for (int i = tid; i < half; i += 256) {
        float s, c;
        sincosf((float)pos * L.freq[i], &s, &c);
        sc[i] = c;
        ss[i] = s;
    }
    T* row = y + (long)t * ld;
    const int hs = L.dp + L.rtp;
    const T* crow = row + (long)L.H * hs;
    float sum = 0.0f;
    for (int j = tid; j < L.rp; j += 256) {
        const float v = to_f(crow[j]);
        sum = fmaf(v, v, sum);
    }
    sum = warp_sum(sum);
    if (lane == 0) sred[warp] = sum;
    __syncthreads();
    float tot = 0.0f;
#pragma unroll
    for (int i = 0; i < 8; i++) tot += sred[i];
    const float inv = 1.0f / sqrtf(tot / (float)L.rank + L.eps);
    T* r1 = ring + (long)(pos % L.cap) * wr;
    T* r2 = keys + (long)(np + t) * wr;
    for (int j = tid; j < L.rp; j += 256) {
        const T v = from_f<T>(to_f(crow[j]) * inv * L.cnorm[j]);
        r1[j] = v;
        r2[j] = v;
    }
    for (int i = tid; i < half; i += 256) {
        const float u = to_f(crow[L.rp + i]), v = to_f(crow[L.rp + i + half]);
        const T a = from_f<T>(u * sc[i] - v * ss[i]), b = from_f<T>(v * sc[i] + u * ss[i]);
        r1[L.rp + i] = a; r1[L.rp + i + half] = b;
        r2[L.rp + i] = a; r2[L.rp + i + half] = b;
    }
    for (int j = L.rot + tid; j < L.rtp; j += 256) {
        r1[L.rp + j] = from_f<T>(0.0f);
        r2[L.rp + j] = from_f<T>(0.0f);
    }
    for (int e = tid; e < L.H * half; e += 256) {
        const int h = e / half, i = e - h * half;
        T* q = row + (long)h * hs + L.dp;
        const float u = to_f(q[i]), v = to_f(q[i + half]);
        q[i] = from_f<T>(u * sc[i] - v * ss[i]);
        q[i + half] = from_f<T>(v * sc[i] + u * ss[i]);
    }
}

// ---------------------------------------------------------------------------- one token

struct StepP {
    const void* y;
    void* ring;
    int* len;
    const void *ukT, *uv;
    void* out;
    float *qa, *qr, *pm, *pl, *pu;    // queries through W_uk^T, rotated parts; per split and head: max, sum, weighted sum
    int splits;
    lt_dn_latent L;
};

// eight lanes per matrix row: dot of a row of n elements with fp32 x in shared memory; the sum in every lane of the eight
template <typename T>
__device__ __forceinline__ float row_dot8(const T* __restrict__ w, const float* x, int n, int g) {
    constexpr int N = Vec<T>::N;
    float a = 0.0f;
#pragma unroll 4
    for (int c = g * N; c < n; c += 8 * N) {
        float f[N];
        Vec<T>::unpack(*(const uint4*)(w + c), f);
#pragma unroll
        for (int i = 0; i < N; i++) a = fmaf(f[i], x[c + i], a);
    }
    a += __shfl_xor_sync(0xffffffffu, a, 1);
    a += __shfl_xor_sync(0xffffffffu, a, 2);
    a += __shfl_xor_sync(0xffffffffu, a, 4);
    return a;
}

// CTA (h, y < ny): 64 rows of q_abs of head h; y = 0 also rotates the head's query.  CTA (0, ny): norms and rotates the
// new row into the ring.
template <typename T>
__global__ void __launch_bounds__(128) k_latent_prep(const __grid_constant__ StepP P) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float sred[4];
    const lt_dn_latent& L = P.L;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int h = blockIdx.x, hs = L.dp + L.rtp, half = L.rot >> 1;
    const int pos = *P.len;
    const T* row = (const T*)P.y;
    if (blockIdx.y == gridDim.y - 1) {
        if (h != 0) return;
        const T* crow = row + (long)L.H * hs;
        T* r = (T*)P.ring + (long)(pos % L.cap) * (L.rp + L.rtp);
        float sum = 0.0f;
        for (int j = tid; j < L.rp; j += 128) {
            const float v = to_f(crow[j]);
            sum = fmaf(v, v, sum);
        }
        sum = warp_sum(sum);
        if (lane == 0) sred[warp] = sum;
        __syncthreads();
        const float inv = 1.0f / sqrtf(((sred[0] + sred[1]) + (sred[2] + sred[3])) / (float)L.rank + L.eps);
        for (int j = tid; j < L.rp; j += 128) r[j] = from_f<T>(to_f(crow[j]) * inv * L.cnorm[j]);
        for (int i = tid; i < half; i += 128) {
            float s, c;
            sincosf((float)pos * L.freq[i], &s, &c);
            const float u = to_f(crow[L.rp + i]), v = to_f(crow[L.rp + i + half]);
            r[L.rp + i] = from_f<T>(u * c - v * s);
            r[L.rp + i + half] = from_f<T>(v * c + u * s);
        }
        for (int j = L.rot + tid; j < L.rtp; j += 128) r[L.rp + j] = from_f<T>(0.0f);
        return;
    }
    const T* q = row + (long)h * hs;
    for (int j = tid; j < L.dp; j += 128) sm[j] = to_f(q[j]);
    if (blockIdx.y == 0) {
        for (int i = tid; i < half; i += 128) {
            float s, c;
            sincosf((float)pos * L.freq[i], &s, &c);
            const float u = to_f(q[L.dp + i]), v = to_f(q[L.dp + i + half]);
            P.qr[h * L.rtp + i] = to_f(from_f<T>(u * c - v * s));
            P.qr[h * L.rtp + i + half] = to_f(from_f<T>(v * c + u * s));
        }
        for (int j = L.rot + tid; j < L.rtp; j += 128) P.qr[h * L.rtp + j] = 0.0f;
    }
    __syncthreads();
    // eight lanes per row of W_uk^T, four rows per group of lanes, all in flight at once
    const int g = tid & 7, r0 = blockIdx.y * 64 + (tid >> 3);
    const T* w = (const T*)P.ukT + (long)h * L.rp * L.dp;
    float a[4] = {0.0f, 0.0f, 0.0f, 0.0f};
    constexpr int N = Vec<T>::N;
    for (int c = g * N; c < L.dp; c += 8 * N) {
        uint4 v[4];
#pragma unroll
        for (int i = 0; i < 4; i++) v[i] = *(const uint4*)(w + (long)min(r0 + 16 * i, L.rp - 1) * L.dp + c);
#pragma unroll
        for (int i = 0; i < 4; i++) {
            float f[N];
            Vec<T>::unpack(v[i], f);
#pragma unroll
            for (int j = 0; j < N; j++) a[i] = fmaf(f[j], sm[c + j], a[i]);
        }
    }
#pragma unroll
    for (int i = 0; i < 4; i++) {
        a[i] += __shfl_xor_sync(0xffffffffu, a[i], 1);
        a[i] += __shfl_xor_sync(0xffffffffu, a[i], 2);
        a[i] += __shfl_xor_sync(0xffffffffu, a[i], 4);
        if (g == 0 && r0 + 16 * i < L.rp) P.qa[h * L.rp + r0 + 16 * i] = a[i];
    }
}

constexpr int SH = 8;      // heads of a CTA
constexpr int SR = 32;     // cache rows staged at a time

template <typename T, int RD>
__global__ void __launch_bounds__(128) k_latent_scan(const __grid_constant__ StepP P) {
    constexpr int N = Vec<T>::N;
    extern __shared__ __align__(16) unsigned char smem[];
    const lt_dn_latent& L = P.L;
    const int wr = L.rp + L.rtp;
    const int units = (wr / N) | 1, stride = units * N;     // odd number of 16-byte units per row
    T* sK = (T*)smem;
    float* sQ = (float*)(smem + (size_t)SR * units * 16);   // [SH][wr]
    __shared__ float sP[SR][SH];
    __shared__ float sF[SH];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int split = blockIdx.x, h0 = blockIdx.y * SH, nh = min(SH, L.H - h0);
    const int pos = *P.len;
    const int n = min(pos + 1, L.window);                   // visible positions: pos - n + 1 .. pos
    const int per = (n + P.splits - 1) / P.splits;
    const int lo = pos - n + 1 + split * per, hi = min(pos + 1, lo + per);

    const int wq = wr >> 2;
    for (int e = tid; e < SH * wq; e += 128) {
        const int h = e / wq, c = (e - h * wq) * 4, hh = h0 + min(h, nh - 1);
        cp16(sQ + h * wr + c, c < L.rp ? P.qa + hh * L.rp + c : P.qr + hh * L.rtp + c - L.rp, h < nh);
    }
    float acc[RD][SH][2];
#pragma unroll
    for (int i = 0; i < RD; i++)
#pragma unroll
        for (int h = 0; h < SH; h++) acc[i][h][0] = acc[i][h][1] = 0.0f;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};   // of the warp's two heads

    for (int p0 = lo; p0 < hi; p0 += SR) {
        const int nr = min(SR, hi - p0);
        const int cu = wr / N;
        __syncthreads();
        for (int e = tid; e < SR * cu; e += 128) {
            const int r = e / cu, c = e - r * cu;
            cp16(sK + r * stride + c * N, (const T*)P.ring + (long)((p0 + min(r, nr - 1)) % L.cap) * wr + c * N, r < nr);
        }
        asm volatile("cp.async.commit_group;\n\tcp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        float s0 = 0.0f, s1 = 0.0f;
        const float* q0 = sQ + (2 * warp) * wr;
        const float* q1 = q0 + wr;
        for (int c = 0; c < wr; c += N) {
            float f[N];
            Vec<T>::unpack(*(const uint4*)(sK + lane * stride + c), f);
#pragma unroll
            for (int i = 0; i < N; i += 4) {
                const float4 a = *(const float4*)(q0 + c + i), b = *(const float4*)(q1 + c + i);
                s0 = fmaf(f[i], a.x, fmaf(f[i + 1], a.y, fmaf(f[i + 2], a.z, fmaf(f[i + 3], a.w, s0))));
                s1 = fmaf(f[i], b.x, fmaf(f[i + 1], b.y, fmaf(f[i + 2], b.z, fmaf(f[i + 3], b.w, s1))));
            }
        }
        const bool ok = lane < nr;
        float s[2] = {ok ? s0 * L.scale : -INFINITY, ok ? s1 * L.scale : -INFINITY};
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const float mx = fmaxf(m[i], warp_max(s[i]));
            const float f = expf(m[i] - mx), p = expf(s[i] - mx);
            m[i] = mx;
            l[i] = l[i] * f + warp_sum(p);
            sP[lane][2 * warp + i] = p;
            if (lane == 0) sF[2 * warp + i] = f;
        }
        __syncthreads();
        float f[SH];
#pragma unroll
        for (int h = 0; h < SH; h++) f[h] = sF[h];
#pragma unroll
        for (int i = 0; i < RD; i++)
#pragma unroll
            for (int h = 0; h < SH; h++) {
                acc[i][h][0] *= f[h];
                acc[i][h][1] *= f[h];
            }
        for (int r = 0; r < nr; r++) {
            const float4 pa = *(const float4*)&sP[r][0], pb = *(const float4*)&sP[r][4];
            const float p[SH] = {pa.x, pa.y, pa.z, pa.w, pb.x, pb.y, pb.z, pb.w};
#pragma unroll
            for (int i = 0; i < RD; i++) {
                const int c = 2 * tid + 256 * i;
                if (c < L.rp) {
                    const float x = to_f(sK[r * stride + c]), y = to_f(sK[r * stride + c + 1]);
#pragma unroll
                    for (int h = 0; h < SH; h++) {
                        acc[i][h][0] = fmaf(p[h], x, acc[i][h][0]);
                        acc[i][h][1] = fmaf(p[h], y, acc[i][h][1]);
                    }
                }
            }
        }
    }
    if (lane == 0) {
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const int h = 2 * warp + i;
            if (h < nh) {
                P.pm[(long)split * L.H + h0 + h] = m[i];
                P.pl[(long)split * L.H + h0 + h] = l[i];
            }
        }
    }
#pragma unroll
    for (int i = 0; i < RD; i++) {
        const int c = 2 * tid + 256 * i;
        if (c < L.rp)
#pragma unroll
            for (int h = 0; h < SH; h++)
                if (h < nh)
                    *(float2*)(P.pu + ((long)split * L.H + h0 + h) * L.rp + c) = make_float2(acc[i][h][0], acc[i][h][1]);
    }
}

// CTA (h, y): combines the splits of head h (two halves of the threads take two halves of the splits), then 32 rows of
// the value projection
constexpr int OT = 256;
template <typename T>
__global__ void __launch_bounds__(OT) k_latent_out(const __grid_constant__ StepP P) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float sred[OT / 32];
    const lt_dn_latent& L = P.L;
    float* su = sm;                // [2][rp]
    float* sw = sm + 2 * L.rp;     // [splits]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.x;
    float m = -INFINITY;
    for (int s = tid; s < P.splits; s += OT) m = fmaxf(m, P.pm[(long)s * L.H + h]);
    m = warp_max(m);
    if (lane == 0) sred[warp] = m;
    __syncthreads();
#pragma unroll
    for (int i = 0; i < OT / 32; i++) m = fmaxf(m, sred[i]);
    __syncthreads();
    float l = 0.0f;
    for (int s = tid; s < P.splits; s += OT) {
        const float w = expf(P.pm[(long)s * L.H + h] - m);
        sw[s] = w;
        l = fmaf(w, P.pl[(long)s * L.H + h], l);
    }
    l = warp_sum(l);
    if (lane == 0) sred[warp] = l;
    __syncthreads();
    l = 0.0f;
#pragma unroll
    for (int i = 0; i < OT / 32; i++) l += sred[i];
    const float inv = 1.0f / l;
    const int half = tid >> 7, hs = (P.splits + 1) >> 1;
    const int s0 = half * hs, s1 = min(P.splits, s0 + hs);
    for (int c = (tid & 127) * 4; c < L.rp; c += 512) {
        const float* u = P.pu + (long)h * L.rp + c;
        float4 a = make_float4(0, 0, 0, 0);
#pragma unroll 8
        for (int s = s0; s < s1; s++) {
            const float4 v = *(const float4*)(u + (long)s * L.H * L.rp);
            const float w = sw[s];
            a.x = fmaf(w, v.x, a.x); a.y = fmaf(w, v.y, a.y); a.z = fmaf(w, v.z, a.z); a.w = fmaf(w, v.w, a.w);
        }
        *(float4*)(su + half * L.rp + c) = make_float4(a.x * inv, a.y * inv, a.z * inv, a.w * inv);
    }
    __syncthreads();
    for (int c = tid; c < L.rp; c += OT) su[c] += su[L.rp + c];
    __syncthreads();
    const int g = tid & 7, v = blockIdx.y * 32 + (tid >> 3);
    const float a = row_dot8<T>((const T*)P.uv + ((long)h * L.dvp + min(v, L.dvp - 1)) * L.rp, su, L.rp, g);
    if (g == 0 && v < L.dvp) ((T*)P.out)[h * L.dvp + v] = from_f<T>(a);
    if (h == 0 && blockIdx.y == 0 && tid == 0) *P.len += 1;     // nothing of this launch reads it
}

template <typename T>
static int launch_step(const StepP& P, cudaStream_t s) {
    const lt_dn_latent& L = P.L;
    const int ny = (L.rp + 63) / 64;
    k_latent_prep<T><<<dim3(L.H, ny + 1), 128, L.dp * 4, s>>>(P);
    int rc = check_launch("lt_dn_latent_step (prep)");
    if (rc != LT_OK) return rc;
    const int wr = L.rp + L.rtp, units = (wr / Vec<T>::N) | 1;
    const size_t smem = (size_t)SR * units * 16 + (size_t)SH * wr * 4;
    LT_REQUIRE(smem <= 220 * 1024, "lt_dn_latent_step: a cache row of %d elements needs %zu bytes of shared memory", wr, smem);
    const dim3 grid(P.splits, (L.H + SH - 1) / SH);
    static PerDeviceOnce once;
    if (once.first()) {
        LT_CUDA(cudaFuncSetAttribute(k_latent_scan<T, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
        LT_CUDA(cudaFuncSetAttribute(k_latent_scan<T, 2>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
        LT_CUDA(cudaFuncSetAttribute(k_latent_scan<T, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
    }
    if (L.rp <= 256) k_latent_scan<T, 1><<<grid, 128, smem, s>>>(P);
    else if (L.rp <= 512) k_latent_scan<T, 2><<<grid, 128, smem, s>>>(P);
    else k_latent_scan<T, 4><<<grid, 128, smem, s>>>(P);
    rc = check_launch("lt_dn_latent_step (scan)");
    if (rc != LT_OK) return rc;
    k_latent_out<T><<<dim3(L.H, (L.dvp + 31) / 32), OT, (2 * L.rp + P.splits) * 4, s>>>(P);
    return check_launch("lt_dn_latent_step (out)");
}

}  // namespace dn
}  // namespace lt

using namespace lt;
using namespace lt::dn;

extern "C" int lt_dn_latent_rows(void* y, int ld, void* ring, void* keys, int np, int pos0, int f32, int T, const lt_dn_latent* h_l,
                                 void* stream) {
    const char* bad = latent_error(h_l);
    LT_REQUIRE(bad == nullptr, "lt_dn_latent_rows: %s", bad);
    LT_REQUIRE(y && ring && keys, "lt_dn_latent_rows: null pointer");
    LT_REQUIRE(T > 0 && np >= 0 && np <= pos0 && np + T <= h_l->cap, "lt_dn_latent_rows: T=%d np=%d pos0=%d do not fit a ring of %d", T, np,
               pos0, h_l->cap);
    const size_t smem = (size_t)(h_l->rot > 0 ? h_l->rot : 2) * 4;
    if (f32) k_latent_rows<float><<<T + np, 256, smem, (cudaStream_t)stream>>>((float*)y, ld, (float*)ring, (float*)keys, np, pos0, T, *h_l);
    else k_latent_rows<bf16><<<T + np, 256, smem, (cudaStream_t)stream>>>((bf16*)y, ld, (bf16*)ring, (bf16*)keys, np, pos0, T, *h_l);
    return check_launch("lt_dn_latent_rows");
}

extern "C" long lt_dn_latent_step_ws(int H, int rp, int rtp, int splits) {
    return (long)H * (rp + rtp) + (long)splits * H * (rp + 2) + 16;
}

extern "C" int lt_dn_latent_step(const void* y, void* ring, int* len, const void* ukT, const void* uv, void* out, int f32,
                                 const lt_dn_latent* h_l, int splits, float* ws, void* stream) {
    const char* bad = latent_error(h_l);
    LT_REQUIRE(bad == nullptr, "lt_dn_latent_step: %s", bad);
    LT_REQUIRE(y && ring && len && ukT && uv && out && ws, "lt_dn_latent_step: null pointer");
    LT_REQUIRE(splits > 0 && splits <= 1024, "lt_dn_latent_step: splits=%d", splits);
    LT_REQUIRE(h_l->rp <= 1024, "lt_dn_latent_step: latent size %d is above 1024", h_l->rp);
    LT_REQUIRE(h_l->cap >= h_l->window, "lt_dn_latent_step: ring of %d rows for a window of %d", h_l->cap, h_l->window);
    LT_REQUIRE(aligned16(y) && aligned16(ring) && aligned16(ukT) && aligned16(uv) && aligned16(ws), "lt_dn_latent_step: pointers must be 16-byte aligned");
    StepP P;
    P.y = y; P.ring = ring; P.len = len; P.ukT = ukT; P.uv = uv; P.out = out; P.splits = splits; P.L = *h_l;
    const long H = h_l->H;
    P.pu = ws;                                 // 8-byte stores: first
    P.qa = P.pu + (long)splits * H * h_l->rp;
    P.qr = P.qa + H * h_l->rp;
    P.pm = P.qr + H * h_l->rtp;
    P.pl = P.pm + (long)splits * H;
    if (f32) return launch_step<float>(P, (cudaStream_t)stream);
    return launch_step<bf16>(P, (cudaStream_t)stream);
}
