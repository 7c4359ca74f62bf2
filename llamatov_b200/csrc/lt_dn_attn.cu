// Softmax attention of a prompt portion over keys and values in memory: k_window_attn is a tiled online softmax on the
// tensor cores (mma.sync m16n8k16, bf16 operands, fp32 accumulation; the softmax weights enter the value product as the sum
// of two bf16), k_window_attn_f32 the fp32 form.  Used with expanded latent keys and values behind a sliding window, and with
// the cache rows of grouped-query attention (no window, capped scores, a gate per head).
#include "lt_dn_gqa.cuh"
#include "lt_dn_latent.cuh"
#include "lt_dn_mma.cuh"

namespace lt {
namespace dn {

struct WinP {
    const void *q, *kn, *kr, *v;
    void* out;
    int ldq, ldkn, ldkr, ldv, ldo, T, np, window, dp, rtp, dvp;
    float scale;
    int per;             // consecutive query heads that share a head of kn and v
    float softcap;       // 0: none
    const float* gate;   // [t][ldg] factors of the heads' outputs, or null
    int ldg;
};

constexpr int WQ = 64, WK = 64;

// CAP: scores pass softcap * tanh(score / softcap)
template <int DV, bool CAP>
__global__ void __launch_bounds__(128) k_window_attn(const __grid_constant__ WinP P) {
    extern __shared__ __align__(16) unsigned char smem[];
    const int DQ = P.dp + P.rtp, DK = (DQ + 15) & ~15;
    const int ks = DK + 8, vs = DV + 8;              // row strides in elements: an odd number of 16-byte units
    bf16* sQ = (bf16*)smem;
    bf16* sK = sQ + WQ * ks;
    bf16* sV = sK + 2 * WK * ks;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int h = blockIdx.y, hk = h / P.per, t0 = (gridDim.x - 1 - blockIdx.x) * WQ, v0 = blockIdx.z * DV;     // longest rows first
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
            const bf16* src = c < c_n ? (const bf16*)P.kn + j * P.ldkn + (long)hk * P.dp + c * 8
                                      : (const bf16*)P.kr + j * P.ldkr + (c - c_n) * 8;
            cp16(k + r * ks + c * 8, src, ok);
        }
        for (int e = tid; e < WK * c_v; e += 128) {
            const int r = e / c_v, c = e - r * c_v;
            const bool ok = j0 + r <= jhi;
            cp16(v + r * vs + c * 8, (const bf16*)P.v + (long)(ok ? j0 + r : 0) * P.ldv + (long)hk * P.dvp + v0 + c * 8, ok);
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
    // softmax weights are powers of two: scores carry a factor log2(e)
    constexpr float LOG2E = 1.4426950408889634f;
    const float sc = CAP ? P.scale * (2.0f * LOG2E) / P.softcap : P.scale * LOG2E, cap = P.softcap * LOG2E;

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
                float x = s[n][i] * sc;
                if (CAP) x = fmaf(-2.0f * cap, __fdividef(1.0f, 1.0f + exp2f(fminf(x, 120.0f))), cap);    // tanh u = 1 - 2 / (1 + e^(2u))
                s[n][i] = see ? x : -INFINITY;
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
        const float inv = (P.gate != nullptr ? P.gate[(long)t * P.ldg + h] : 1.0f) / l[r];
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
    const int t = blockIdx.x, h = blockIdx.y, hk = h / P.per;
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
            const float* kn = (const float*)P.kn + (long)j * P.ldkn + (long)hk * P.dp;
            const float* kr = (const float*)P.kr + (long)j * P.ldkr;
            float a = 0.0f;
            for (int c = 0; c < P.dp; c++) a = fmaf(sq[c], kn[c], a);
            for (int c = 0; c < P.rtp; c++) a = fmaf(sq[P.dp + c], kr[c], a);
            s = a * P.scale;
            if (P.softcap > 0.0f) s = P.softcap * tanhf(s / P.softcap);
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
                    a = fmaf(sp[jj], ((const float*)P.v)[(long)(j0 + jj) * P.ldv + (long)hk * P.dvp + c], a);
                o[i] = a;
            }
        }
        __syncthreads();
    }
    const float gate = P.gate != nullptr ? P.gate[(long)t * P.ldg + h] : 1.0f;
#pragma unroll
    for (int i = 0; i < 8; i++) {
        const int c = tid + i * 128;
        if (c < P.dvp) ((float*)P.out)[(long)t * P.ldo + (long)h * P.dvp + c] = o[i] / l * gate;
    }
}

template <int DV, bool CAP>
static int launch_window(const WinP& P, int H, cudaStream_t s) {
    const int DK = (P.dp + P.rtp + 15) & ~15;
    const size_t smem = (size_t)((WQ + 2 * WK) * (DK + 8) + 2 * WK * (DV + 8)) * 2;
    LT_REQUIRE(smem <= 220 * 1024, "attention of a portion: key size %d needs %zu bytes of shared memory", P.dp + P.rtp, smem);
    static PerDeviceOnce once;
    if (once.first())
        LT_CUDA(cudaFuncSetAttribute(k_window_attn<DV, CAP>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
    k_window_attn<DV, CAP><<<dim3((P.T + WQ - 1) / WQ, H, (P.dvp + DV - 1) / DV), 128, smem, s>>>(P);
    return check_launch("attention of a portion");
}

template <bool CAP>
static int launch_dv(const WinP& P, int H, cudaStream_t s) {
    if (P.dvp <= 32) return launch_window<32, CAP>(P, H, s);
    if (P.dvp <= 64) return launch_window<64, CAP>(P, H, s);
    return launch_window<128, CAP>(P, H, s);
}
static int launch_attn(const WinP& P, int f32, int H, cudaStream_t s) {
    if (f32) {
        LT_REQUIRE(P.dvp <= 1024 && P.dp + P.rtp <= 8192, "attention of a portion: head sizes %d, %d", P.dp + P.rtp, P.dvp);
        k_window_attn_f32<<<dim3(P.T, H), 128, (P.dp + P.rtp + 128) * 4, s>>>(P);
        return check_launch("attention of a portion");
    }
    return P.softcap > 0.0f ? launch_dv<true>(P, H, s) : launch_dv<false>(P, H, s);
}

}  // namespace dn
}  // namespace lt

using namespace lt;
using namespace lt::dn;

extern "C" int lt_dn_window_attn(const void* q, int ldq, const void* kn, int ldkn, const void* kr, int ldkr, const void* v, int ldv,
                                 void* out, int ldo, int f32, int T, int np, const lt_dn_latent* h_l, void* stream) {
    const char* bad = latent_error(h_l);
    LT_REQUIRE(bad == nullptr, "lt_dn_window_attn: %s", bad);
    LT_REQUIRE(q && kn && kr && v && out && T > 0 && np >= 0, "lt_dn_window_attn: null pointer or T=%d np=%d", T, np);
    LT_REQUIRE(ldq % 8 == 0 && ldkn % 8 == 0 && ldkr % 8 == 0 && ldv % 8 == 0 && ldo % 8 == 0, "lt_dn_window_attn: row strides must be multiples of 8");
    LT_REQUIRE(aligned16(q) && aligned16(kn) && aligned16(kr) && aligned16(v) && aligned16(out), "lt_dn_window_attn: pointers must be 16-byte aligned");
    WinP P = {q, kn, kr, v, out, ldq, ldkn, ldkr, ldv, ldo, T, np, h_l->window, h_l->dp, h_l->rtp, h_l->dvp, h_l->scale};
    P.per = 1;
    return launch_attn(P, f32, h_l->H, (cudaStream_t)stream);
}

extern "C" int lt_dn_gqa_attn(const void* q, int ldq, const void* kc, const void* vc, const float* gate, int ldg, void* out, int ldo,
                              int f32, int T, int np, const lt_dn_gqa* h_a, void* stream) {
    const char* bad = gqa_error(h_a);
    LT_REQUIRE(bad == nullptr, "lt_dn_gqa_attn: %s", bad);
    LT_REQUIRE(q && kc && vc && out && T > 0 && np >= 0 && np + T <= h_a->cap, "lt_dn_gqa_attn: null pointer or T=%d np=%d", T, np);
    LT_REQUIRE(ldq % 8 == 0 && ldo % 8 == 0 && aligned16(q) && aligned16(kc) && aligned16(vc) && aligned16(out),
               "lt_dn_gqa_attn: row strides must be multiples of 8, pointers 16-byte aligned");
    const int ldk = h_a->G * h_a->dp, ldv = h_a->G * h_a->dvp;
    WinP P = {q, kc, nullptr, vc, out, ldq, ldk, 0, ldv, ldo, T, np, INT_MAX, h_a->dp, 0, h_a->dvp, h_a->scale};
    P.per = h_a->H / h_a->G;
    P.softcap = h_a->softcap;
    P.gate = gate;
    P.ldg = ldg;
    return launch_attn(P, f32, h_a->H, (cudaStream_t)stream);
}
