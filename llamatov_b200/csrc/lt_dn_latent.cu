// Windowed attention over a latent cache: per position one row [c, kr], c the normed latent that keys and values of
// every head are projections of, kr the rotated key part the heads share.
//
// Prompt portions (lt_dn_latent_rows, then the key/value expansion by lt_dn_linear, then lt_dn_window_attn): keys and
// values of the portion and of the window before it are expanded per head; k_window_attn is a tiled online softmax on
// the tensor cores (mma.sync m16n8k16, bf16 operands, fp32 accumulation; the softmax weights enter the value product
// as the sum of two bf16), k_window_attn_f32 the fp32 form.
// One token (lt_dn_latent_step, three launches): nothing is expanded.  The query is taken through W_uk^T, scores and
// the weighted sum are over the latent rows (all heads read the same rows), and the value projection is applied to the
// sum.
#include "lt_dn_common.cuh"

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

// ---------------------------------------------------------------------------- window attention of a portion

struct WinP {
    const void *q, *kn, *kr, *v;
    void* out;
    int ldq, ldkn, ldkr, ldv, ldo, T, np, window, dp, rtp, dvp;
    float scale;
};

__device__ __forceinline__ unsigned s_u32(const void* p) { return (unsigned)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp16(void* dst, const void* src, bool ok) {
    const int n = ok ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(s_u32(dst)), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void ldsm4(unsigned (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(s_u32(p))
                 : "memory");
}
__device__ __forceinline__ void ldsm4t(unsigned (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(s_u32(p))
                 : "memory");
}
__device__ __forceinline__ void mma16816(float (&d)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// (x, y) as packed bf16 plus the packed remainders: hi + lo carries 16 significant bits
__device__ __forceinline__ void split2(float x, float y, unsigned& hi, unsigned& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
    hi = *(const unsigned*)&h;
    lo = *(const unsigned*)&l;
}

constexpr int WQ = 64, WK = 64;

template <int DV>
__global__ void __launch_bounds__(128) k_window_attn(const __grid_constant__ WinP P) {
    extern __shared__ __align__(16) unsigned char smem[];
    const int DQ = P.dp + P.rtp, DK = (DQ + 15) & ~15;
    const int ks = DK + 8, vs = DV + 8;              // row strides in elements: an odd number of 16-byte units
    bf16* sQ = (bf16*)smem;
    bf16* sK = sQ + WQ * ks;
    bf16* sV = sK + 2 * WK * ks;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int h = blockIdx.y, t0 = (gridDim.x - 1 - blockIdx.x) * WQ, v0 = blockIdx.z * DV;     // longest rows first
    const int c_n = P.dp >> 3, c_r = P.rtp >> 3, c_v = (min(DV, P.dvp - v0)) >> 3;
    const int qlast = min(t0 + WQ, P.T) - 1;
    const int jlo = max(0, P.np + t0 - P.window + 1), jhi = P.np + qlast;   // keys any query of the tile sees

    // columns no copy writes
    for (int e = tid; e < WQ * (DK - DQ) / 8; e += 128) *(uint4*)(sQ + e * ks + DQ) = make_uint4(0, 0, 0, 0);
    for (int e = tid; e < 2 * WK * (DK - DQ) / 8; e += 128) *(uint4*)(sK + e * ks + DQ) = make_uint4(0, 0, 0, 0);
    for (int e = tid; e < 2 * WK * (DV / 8 - c_v); e += 128)
        *(uint4*)(sV + (e / (DV / 8 - c_v)) * vs + (c_v + e % (DV / 8 - c_v)) * 8) = make_uint4(0, 0, 0, 0);

    const int cq = c_n + c_r;
    for (int e = tid; e < WQ * cq; e += 128) {
        const int r = e / cq, c = e - r * cq;
        const bool ok = t0 + r < P.T;
        cp16(sQ + r * ks + c * 8, (const bf16*)P.q + (long)(ok ? t0 + r : 0) * P.ldq + (long)h * DQ + c * 8, ok);
    }
    auto load_kv = [&](int j0, int b) {
        bf16* k = sK + b * WK * ks;
        bf16* v = sV + b * WK * vs;
        for (int e = tid; e < WK * cq; e += 128) {
            const int r = e / cq, c = e - r * cq;
            const bool ok = j0 + r <= jhi;
            const long j = ok ? j0 + r : 0;
            const bf16* src = c < c_n ? (const bf16*)P.kn + j * P.ldkn + (long)h * P.dp + c * 8
                                      : (const bf16*)P.kr + j * P.ldkr + (c - c_n) * 8;
            cp16(k + r * ks + c * 8, src, ok);
        }
        for (int e = tid; e < WK * c_v; e += 128) {
            const int r = e / c_v, c = e - r * c_v;
            const bool ok = j0 + r <= jhi;
            cp16(v + r * vs + c * 8, (const bf16*)P.v + (long)(ok ? j0 + r : 0) * P.ldv + (long)h * P.dvp + v0 + c * 8, ok);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load_kv(jlo, 0);

    const int g = lane >> 2, tg = lane & 3;
    const int q0 = P.np + t0 + warp * 16 + g;        // key index of this thread's two query rows: q0, q0 + 8
    float o[DV / 8][4];
#pragma unroll
    for (int i = 0; i < DV / 8; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
    const float sc = P.scale * 1.4426950408889634f;

    int b = 0;
    for (int j0 = jlo; j0 <= jhi; j0 += WK, b ^= 1) {
        if (j0 + WK <= jhi) {
            load_kv(j0 + WK, b ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const bf16* k = sK + b * WK * ks;
        const bf16* v = sV + b * WK * vs;
        float s[8][4];
#pragma unroll
        for (int i = 0; i < 8; i++) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.0f;
        for (int kk = 0; kk < DK; kk += 16) {
            unsigned a[4];
            ldsm4(a, sQ + (warp * 16 + (lane & 15)) * ks + kk + (lane >> 4) * 8);
#pragma unroll
            for (int n = 0; n < 8; n += 2) {
                unsigned r[4];
                ldsm4(r, k + (n * 8 + (lane & 7) + ((lane >> 4) << 3)) * ks + kk + ((lane >> 3) & 1) * 8);
                mma16816(s[n], a, r[0], r[1]);
                mma16816(s[n + 1], a, r[2], r[3]);
            }
        }
        // mask, running maximum
        float mx[2] = {m[0], m[1]};
#pragma unroll
        for (int n = 0; n < 8; n++)
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const int j = j0 + n * 8 + tg * 2 + (i & 1), q = q0 + (i >> 1) * 8;
                const bool see = j <= q && q - j < P.window;
                s[n][i] = see ? s[n][i] * sc : -INFINITY;
                mx[i >> 1] = fmaxf(mx[i >> 1], s[n][i]);
            }
#pragma unroll
        for (int r = 0; r < 2; r++) {
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
            const float base = mx[r] == -INFINITY ? 0.0f : mx[r];
            const float f = exp2f(m[r] - base);      // 0 when nothing has been seen yet
            m[r] = mx[r];
            l[r] *= f;
#pragma unroll
            for (int i = 0; i < DV / 8; i++) {
                o[i][2 * r] *= f;
                o[i][2 * r + 1] *= f;
            }
#pragma unroll
            for (int n = 0; n < 8; n++) {
                s[n][2 * r] = exp2f(s[n][2 * r] - base);
                s[n][2 * r + 1] = exp2f(s[n][2 * r + 1] - base);
                l[r] += s[n][2 * r] + s[n][2 * r + 1];
            }
        }
#pragma unroll
        for (int kk = 0; kk < 4; kk++) {
            unsigned hi[4], lo[4];
            split2(s[2 * kk][0], s[2 * kk][1], hi[0], lo[0]);
            split2(s[2 * kk][2], s[2 * kk][3], hi[1], lo[1]);
            split2(s[2 * kk + 1][0], s[2 * kk + 1][1], hi[2], lo[2]);
            split2(s[2 * kk + 1][2], s[2 * kk + 1][3], hi[3], lo[3]);
#pragma unroll
            for (int n = 0; n < DV / 8; n += 2) {
                unsigned r[4];
                ldsm4t(r, v + (kk * 16 + (lane & 15)) * vs + n * 8 + (lane >> 4) * 8);
                mma16816(o[n], hi, r[0], r[1]);
                mma16816(o[n], lo, r[0], r[1]);
                mma16816(o[n + 1], hi, r[2], r[3]);
                mma16816(o[n + 1], lo, r[2], r[3]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int r = 0; r < 2; r++) {
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
        const int t = t0 + warp * 16 + g + r * 8;
        if (t >= P.T) continue;
        const float inv = 1.0f / l[r];
        bf16* out = (bf16*)P.out + (long)t * P.ldo + (long)h * P.dvp;
#pragma unroll
        for (int n = 0; n < DV / 8; n++) {
            const int c = v0 + n * 8 + tg * 2;
            if (c < P.dvp) *(__nv_bfloat162*)(out + c) = __floats2bfloat162_rn(o[n][2 * r] * inv, o[n][2 * r + 1] * inv);
        }
    }
}

// one (query, head) per CTA, 128 keys at a time
__global__ void __launch_bounds__(128) k_window_attn_f32(const __grid_constant__ WinP P) {
    extern __shared__ __align__(16) float smf[];
    const int DQ = P.dp + P.rtp, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    float* sq = smf;
    float* sp = sq + DQ;        // 128 weights
    __shared__ float sred[4];
    const int t = blockIdx.x, h = blockIdx.y;
    const float* q = (const float*)P.q + (long)t * P.ldq + (long)h * DQ;
    for (int j = tid; j < DQ; j += 128) sq[j] = q[j];
    const int qi = P.np + t, jlo = max(0, qi - P.window + 1);
    float m = -INFINITY, l = 0.0f, o[8];
#pragma unroll
    for (int i = 0; i < 8; i++) o[i] = 0.0f;
    __syncthreads();
    for (int j0 = jlo; j0 <= qi; j0 += 128) {
        const int j = j0 + tid;
        float s = -INFINITY;
        if (j <= qi) {
            const float* kn = (const float*)P.kn + (long)j * P.ldkn + (long)h * P.dp;
            const float* kr = (const float*)P.kr + (long)j * P.ldkr;
            float a = 0.0f;
            for (int c = 0; c < P.dp; c++) a = fmaf(sq[c], kn[c], a);
            for (int c = 0; c < P.rtp; c++) a = fmaf(sq[P.dp + c], kr[c], a);
            s = a * P.scale;
        }
        float mx = warp_max(s);
        if (lane == 0) sred[warp] = mx;
        __syncthreads();
        mx = fmaxf(fmaxf(fmaxf(sred[0], sred[1]), fmaxf(sred[2], sred[3])), m);
        const float f = expf(m - mx), p = expf(s - mx);      // a chunk always has a visible key: mx is finite
        m = mx;
        sp[tid] = p;
        float ps = warp_sum(p);
        __syncthreads();
        if (lane == 0) sred[warp] = ps;
        __syncthreads();
        l = l * f + (sred[0] + sred[1]) + (sred[2] + sred[3]);
        const int n = min(128, qi - j0 + 1);
#pragma unroll
        for (int i = 0; i < 8; i++) {
            const int c = tid + i * 128;
            if (c < P.dvp) {
                float a = o[i] * f;
                for (int jj = 0; jj < n; jj++)
                    a = fmaf(sp[jj], ((const float*)P.v)[(long)(j0 + jj) * P.ldv + (long)h * P.dvp + c], a);
                o[i] = a;
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 8; i++) {
        const int c = tid + i * 128;
        if (c < P.dvp) ((float*)P.out)[(long)t * P.ldo + (long)h * P.dvp + c] = o[i] / l;
    }
}

template <int DV>
static int launch_window(const WinP& P, int H, cudaStream_t s) {
    const int DK = (P.dp + P.rtp + 15) & ~15;
    const size_t smem = (size_t)((WQ + 2 * WK) * (DK + 8) + 2 * WK * (DV + 8)) * 2;
    LT_REQUIRE(smem <= 220 * 1024, "lt_dn_window_attn: key size %d needs %zu bytes of shared memory", P.dp + P.rtp, smem);
    static PerDeviceOnce once;
    if (once.first())
        LT_CUDA(cudaFuncSetAttribute(k_window_attn<DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
    k_window_attn<DV><<<dim3((P.T + WQ - 1) / WQ, H, (P.dvp + DV - 1) / DV), 128, smem, s>>>(P);
    return check_launch("lt_dn_window_attn");
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

static const char* latent_error(const lt_dn_latent* L) {
    if (L == nullptr) return "null description";
    if (L->H <= 0 || L->dp < 0 || L->rtp < 0 || L->dvp <= 0 || L->rp <= 0) return "sizes must be positive";
    if (L->dp % 8 || L->rtp % 8 || L->dvp % 8 || L->rp % 8) return "padded sizes must be multiples of 8";
    if (L->rot < 0 || L->rot % 2 || L->rot > L->rtp) return "rotated dimensions must be even and fit their padded size";
    if (L->rank <= 0 || L->rank > L->rp) return "latent size";
    if (L->window <= 0 || L->cap <= 0) return "window and ring must be positive";
    if (L->cnorm == nullptr || (L->rot > 0 && L->freq == nullptr)) return "null constants";
    return nullptr;
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

extern "C" int lt_dn_window_attn(const void* q, int ldq, const void* kn, int ldkn, const void* kr, int ldkr, const void* v, int ldv,
                                 void* out, int ldo, int f32, int T, int np, const lt_dn_latent* h_l, void* stream) {
    const char* bad = latent_error(h_l);
    LT_REQUIRE(bad == nullptr, "lt_dn_window_attn: %s", bad);
    LT_REQUIRE(q && kn && kr && v && out && T > 0 && np >= 0, "lt_dn_window_attn: null pointer or T=%d np=%d", T, np);
    LT_REQUIRE(ldq % 8 == 0 && ldkn % 8 == 0 && ldkr % 8 == 0 && ldv % 8 == 0 && ldo % 8 == 0, "lt_dn_window_attn: row strides must be multiples of 8");
    LT_REQUIRE(aligned16(q) && aligned16(kn) && aligned16(kr) && aligned16(v) && aligned16(out), "lt_dn_window_attn: pointers must be 16-byte aligned");
    WinP P = {q, kn, kr, v, out, ldq, ldkn, ldkr, ldv, ldo, T, np, h_l->window, h_l->dp, h_l->rtp, h_l->dvp, h_l->scale};
    cudaStream_t s = (cudaStream_t)stream;
    if (f32) {
        LT_REQUIRE(h_l->dvp <= 1024 && h_l->dp + h_l->rtp <= 8192, "lt_dn_window_attn: head sizes %d, %d", h_l->dp + h_l->rtp, h_l->dvp);
        k_window_attn_f32<<<dim3(T, h_l->H), 128, (h_l->dp + h_l->rtp + 128) * 4, s>>>(P);
        return check_launch("lt_dn_window_attn");
    }
    if (h_l->dvp <= 32) return launch_window<32>(P, h_l->H, s);
    if (h_l->dvp <= 64) return launch_window<64>(P, h_l->H, s);
    return launch_window<128>(P, h_l->H, s);
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
