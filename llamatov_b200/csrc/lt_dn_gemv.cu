// Linear for one token, y[n] = epilogue(sum_k W[n][k] x[k]), with the input made where it is used: every CTA turns
// the fp32 vector into the matrix's element type itself (cast, RMS norm over groups, gate), so that norm, gate and
// linear are one launch.  A warp owns pairs of rows (n, n + 1; gate n and its up row; or the one kind, then the other) and keeps two rows x U 16-byte
// loads per lane in flight; the first batch of weights is requested before the input is touched.
#include "lt_dn_common.cuh"

namespace lt {
namespace dn {

struct GemvP {
    const void* W;
    void* Y;
    int M, K, ldw, npair;
    int nstore, mstore;      // pairs of stored rows and those rows; the pairs that follow are gate and up
    lt_dn_prologue pro;
    lt_dn_epilogue epi;
};

constexpr int GV_THREADS = 256;
constexpr int GV_U = 4;

// x as float4 quads in shared memory, those of even index first: the lanes of a warp, 8 elements apart, then read
// consecutive 16-byte words
template <typename T>
__device__ __forceinline__ int quad_slot(int q, int nquad) {
    return Vec<T>::N == 8 ? (q & 1) * (nquad >> 1) + (q >> 1) : q;
}
template <typename T>
__device__ __forceinline__ void put_x(float4* xs, int nquad, int q, float4 v) {
    v.x = to_f(from_f<T>(v.x)); v.y = to_f(from_f<T>(v.y)); v.z = to_f(from_f<T>(v.z)); v.w = to_f(from_f<T>(v.w));
    xs[quad_slot<T>(q, nquad)] = v;
}
template <typename T>
__device__ __forceinline__ float4 load4(const void* p, int q) {
    if (sizeof(T) == 4) return ((const float4*)p)[q];
    const uint2 r = ((const uint2*)p)[q];
    return make_float4(lo_f(r.x), hi_f(r.x), lo_f(r.y), hi_f(r.y));
}

template <typename T>
__device__ __forceinline__ void make_input(const lt_dn_prologue& p, int K, float4* xs, float* sred) {
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int nquad = K >> 2;
    if (p.kind == LT_DN_IN_TYPED) {
        for (int q = tid; q < nquad; q += GV_THREADS) put_x<T>(xs, nquad, q, load4<T>(p.x, q));
        return;
    }
    if (p.kind == LT_DN_IN_CAST) {
        const int q1 = p.n1 >> 2;
        for (int q = tid; q < nquad; q += GV_THREADS)
            put_x<T>(xs, nquad, q, q < q1 ? ((const float4*)p.x)[q] : ((const float4*)p.x2)[q - q1]);
        return;
    }
    const int n1 = p.n1 > 0 ? p.n1 : K, nq1 = n1 >> 2;
    for (int q = nq1 + tid; q < nquad; q += GV_THREADS) put_x<T>(xs, nquad, q, load4<T>(p.x2, q - nq1));
    const bool gf = p.gate_first;
    if (p.seg > 0) {             // groups that do not follow the padded segments: element by element
        const int ng = n1 / p.segp * p.seg / p.count;
        float* inv = (float*)(xs + nquad);
        auto in1 = [&](int j) { return ((const float*)p.x)[j] * (gf ? to_f(((const T*)p.gate)[j]) : 1.0f); };
        for (int g = warp; g < ng; g += GV_THREADS / 32) {
            float s = 0.0f;
            for (int r = g * p.count + lane; r < (g + 1) * p.count; r += 32) {
                const float v = in1(r / p.seg * p.segp + r % p.seg);
                s = fmaf(v, v, s);
            }
            s = warp_sum(s);
            if (lane == 0) inv[g] = 1.0f / sqrtf(s / (float)p.count + p.eps);
        }
        __syncthreads();
        for (int q = tid; q < nq1; q += GV_THREADS) {
            float o[4];
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const int j = 4 * q + i, r = j % p.segp;
                o[i] = 0.0f;
                if (r < p.seg) {
                    o[i] = in1(j) * inv[(j / p.segp * p.seg + r) / p.count] * p.w[j];
                    if (p.gate != nullptr && !gf) o[i] *= to_f(((const T*)p.gate)[j]);
                }
            }
            put_x<T>(xs, nquad, q, make_float4(o[0], o[1], o[2], o[3]));
        }
        return;
    }
    const int gq = p.group >> 2, ng = n1 / p.group, wq = p.w_period >> 2;
    auto in4 = [&](int q) {      // what the norm sees
        float4 v = ((const float4*)p.x)[q];
        if (gf) {
            const float4 g = load4<T>(p.gate, q);
            v.x *= g.x; v.y *= g.y; v.z *= g.z; v.w *= g.w;
        }
        return v;
    };
    auto emit = [&](int q, float4 v, float inv) {
        const float4 w = ((const float4*)p.w)[q % wq];
        v.x = v.x * inv * w.x; v.y = v.y * inv * w.y; v.z = v.z * inv * w.z; v.w = v.w * inv * w.w;
        if (p.gate != nullptr && !gf) {
            const float4 g = load4<T>(p.gate, q);
            v.x *= g.x; v.y *= g.y; v.z *= g.z; v.w *= g.w;
        }
        put_x<T>(xs, nquad, q, v);
    };
    if (ng == 1) {      // one group: the whole CTA
        float s = 0.0f;
        for (int q = tid; q < nq1; q += GV_THREADS) {
            const float4 v = in4(q);
            s = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, s))));
        }
        s = warp_sum(s);
        if (lane == 0) sred[warp] = s;
        __syncthreads();
        float tot = 0.0f;
#pragma unroll
        for (int i = 0; i < GV_THREADS / 32; i++) tot += sred[i];
        const float inv = 1.0f / sqrtf(tot / (float)p.count + p.eps);
        for (int q = tid; q < nq1; q += GV_THREADS) emit(q, in4(q), inv);
    } else {            // many groups: a warp each
        for (int g = warp; g < ng; g += GV_THREADS / 32) {
            float s = 0.0f;
            for (int q = lane; q < gq; q += 32) {
                const float4 v = in4(g * gq + q);
                s = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, s))));
            }
            s = warp_sum(s);
            const float inv = 1.0f / sqrtf(s / (float)p.count + p.eps);
            for (int q = lane; q < gq; q += 32) emit(g * gq + q, in4(g * gq + q), inv);
        }
    }
}

template <typename T>
__global__ void __launch_bounds__(GV_THREADS, 2) k_gemv(const __grid_constant__ GemvP P) {
    extern __shared__ __align__(16) float4 xs[];
    __shared__ float sred[GV_THREADS / 32];
    constexpr int N = Vec<T>::N;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int nvec = P.K / N, nquad = P.K >> 2;
    const int gw = blockIdx.x * (GV_THREADS / 32) + warp, nw = gridDim.x * (GV_THREADS / 32);
    const uint4 zero = make_uint4(0, 0, 0, 0);

    uint4 buf[2][GV_U];
    auto rows_of = [&](int pr, int& r0, int& r1) {
        if (pr >= P.nstore) {
            r0 = P.mstore + pr - P.nstore;
            r1 = r0 + P.npair - P.nstore;
        } else {
            r0 = 2 * pr;
            r1 = r0 + 1 < P.mstore ? r0 + 1 : r0;
        }
    };
    auto fetch = [&](int r0, int r1, int base) {
        const uint4* a = (const uint4*)((const T*)P.W + (long)r0 * P.ldw);
        const uint4* b = (const uint4*)((const T*)P.W + (long)r1 * P.ldw);
#pragma unroll
        for (int u = 0; u < GV_U; u++) {
            const int i = base + u * 32 + lane;
            const bool ok = i < nvec;
            int4 va = make_int4(0, 0, 0, 0), vb = va;
            if (ok) {
                va = ld_stream_v4(a + i);
                vb = ld_stream_v4(b + i);
            }
            buf[0][u] = ok ? make_uint4(va.x, va.y, va.z, va.w) : zero;
            buf[1][u] = ok ? make_uint4(vb.x, vb.y, vb.z, vb.w) : zero;
        }
    };
    int pr = gw, r0 = 0, r1 = 0;
    if (pr < P.npair) {
        rows_of(pr, r0, r1);
        fetch(r0, r1, 0);
    }
    make_input<T>(P.pro, P.K, xs, sred);
    __syncthreads();

    for (; pr < P.npair; pr += nw) {
        float acc0 = 0.0f, acc1 = 0.0f;
        const int c0 = r0, c1 = r1;
        for (int base = 0; base < nvec; base += 32 * GV_U) {
            uint4 w[2][GV_U];
#pragma unroll
            for (int u = 0; u < GV_U; u++) {
                w[0][u] = buf[0][u];
                w[1][u] = buf[1][u];
            }
            if (base + 32 * GV_U < nvec) fetch(c0, c1, base + 32 * GV_U);
            else if (pr + nw < P.npair) {
                rows_of(pr + nw, r0, r1);
                fetch(r0, r1, 0);
            }
#pragma unroll
            for (int u = 0; u < GV_U; u++) {
                const int i = base + u * 32 + lane;
                if (i >= nvec) continue;
                float f0[N], f1[N], x[N];
                Vec<T>::unpack(w[0][u], f0);
                Vec<T>::unpack(w[1][u], f1);
#pragma unroll
                for (int j = 0; j < N / 4; j++) {
                    const float4 q = xs[N == 8 ? j * (nquad >> 1) + i : i];
                    x[4 * j] = q.x; x[4 * j + 1] = q.y; x[4 * j + 2] = q.z; x[4 * j + 3] = q.w;
                }
#pragma unroll
                for (int j = 0; j < N; j++) {
                    acc0 = fmaf(f0[j], x[j], acc0);
                    acc1 = fmaf(f1[j], x[j], acc1);
                }
            }
        }
        acc0 = warp_sum(acc0);
        acc1 = warp_sum(acc1);
        if (pr >= P.nstore) {
            if (lane == 0) glu_store<T>(P.epi, P.epi.kind == LT_DN_GLU ? P.Y : P.epi.y2, c0 - P.mstore, acc0, acc1);
        } else if (lane < 2 && (lane == 0 || c1 != c0)) {
            const int n = lane == 0 ? c0 : c1;
            epi_store<T>(P.epi, row_epi(P.epi, n), P.Y, 0, 0, n, lane == 0 ? acc0 : acc1);
        }
    }
}

}  // namespace dn
}  // namespace lt

using namespace lt;
using namespace lt::dn;

extern "C" int lt_dn_gemv(const void* W, int ldw, void* Y, int f32, int M, int K, const lt_dn_prologue* h_pro,
                          const lt_dn_epilogue* h_epi, void* stream) {
    LT_REQUIRE(W && Y && h_pro, "lt_dn_gemv: null pointer");
    const char* bad = epi_error(h_epi);
    LT_REQUIRE(bad == nullptr, "lt_dn_gemv: %s", bad);
    LT_REQUIRE(M > 0 && K > 0 && K % 8 == 0 && ldw >= K && ldw % 8 == 0, "lt_dn_gemv: M=%d K=%d ldw=%d (multiples of 8)", M, K, ldw);
    LT_REQUIRE(aligned16(W) && aligned16(h_pro->x), "lt_dn_gemv: pointers must be 16-byte aligned");
    const lt_dn_prologue& p = *h_pro;
    LT_REQUIRE(p.x != nullptr, "lt_dn_gemv: null input");
    if (p.kind == LT_DN_IN_CAST)
        LT_REQUIRE(p.n1 % 4 == 0 && p.n1 > 0 && p.n1 <= K && (p.n1 == K || p.x2 != nullptr), "lt_dn_gemv: n1=%d", p.n1);
    int ragged = 0;
    if (p.kind == LT_DN_IN_NORM) {
        const int n1 = p.n1 > 0 ? p.n1 : K;
        LT_REQUIRE(n1 <= K && n1 % 8 == 0 && (n1 == K || (p.x2 != nullptr && aligned16(p.x2))), "lt_dn_gemv: n1=%d of K=%d", n1, K);
        LT_REQUIRE(p.w && p.count > 0 && p.w_period > 0 && p.w_period % 4 == 0 && (!p.gate_first || p.gate != nullptr),
                   "lt_dn_gemv: norm count=%d w_period=%d", p.count, p.w_period);
        if (p.seg > 0) {
            LT_REQUIRE(p.segp >= p.seg && n1 % p.segp == 0 && (n1 / p.segp * p.seg) % p.count == 0 && p.w_period >= n1,
                       "lt_dn_gemv: norm segments of %d in %d, groups of %d", p.seg, p.segp, p.count);
            ragged = n1 / p.segp * p.seg / p.count;
        } else {
            LT_REQUIRE(p.group > 0 && p.group % 4 == 0 && n1 % p.group == 0, "lt_dn_gemv: norm group=%d of %d", p.group, n1);
        }
    }
    const size_t smem = (size_t)K * 4 + (size_t)ragged * 4;
    LT_REQUIRE(smem <= 200 * 1024, "lt_dn_gemv: K=%d needs %zu bytes of shared memory", K, smem);
    GemvP P;
    P.W = W; P.Y = Y; P.M = M; P.K = K; P.ldw = ldw; P.pro = p; P.epi = *h_epi;
    P.mstore = h_epi->kind == LT_DN_GLU ? 0 : M;
    if (h_epi->kind == LT_DN_STORE_GLU) {
        LT_REQUIRE(h_epi->glu_from > 0 && h_epi->glu_from < M && h_epi->y2 != nullptr, "lt_dn_gemv: glu_from=%d of %d outputs", h_epi->glu_from, M);
        P.mstore = h_epi->glu_from;
    }
    P.nstore = (P.mstore + 1) / 2;
    P.npair = P.nstore + M - P.mstore;
    static PerDeviceOnce once;
    if (once.first()) {
        LT_CUDA(cudaFuncSetAttribute(k_gemv<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
        LT_CUDA(cudaFuncSetAttribute(k_gemv<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    }
    const int per = smem <= 100 * 1024 ? 2 : 1;
    const int need = (P.npair + GV_THREADS / 32 - 1) / (GV_THREADS / 32);
    const int grid = need < per * sm_count() ? need : per * sm_count();
    if (f32) k_gemv<float><<<grid, GV_THREADS, smem, (cudaStream_t)stream>>>(P);
    else k_gemv<bf16><<<grid, GV_THREADS, smem, (cudaStream_t)stream>>>(P);
    return check_launch("lt_dn_gemv");
}
