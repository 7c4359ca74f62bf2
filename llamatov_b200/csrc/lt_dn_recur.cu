// Linear-attention recurrence with decay, S <- diag(a_t) S + k_t v_t^T, o_t = S^T q_t, state in fp32; the state-space form
// (DEC_HEAD) has a decay and a step size per token and head, S <- a_t S + dt_t k_t v_t^T, o_t = S^T q_t + D v_t.
//
// k_recur_scan walks the tokens in order (decode, fp32, short portions): a CTA owns 32 value columns of one head,
// eight lanes share a column (dp/8 key channels each, in registers), q, k and the decays are staged 16 tokens at a time.
#include "lt_dn_common.cuh"

namespace lt {
namespace dn {

struct RecurP {
    const void *q, *k, *v;
    float *S, *o;
    int ld, ldo, T, H, dp, dvp, per;     // per: consecutive heads that share q and k
    lt_dn_decay dec;
};

enum { DEC_CONST = 0, DEC_LOG = 1, DEC_LOWRANK = 2, DEC_HEAD = 3 };
constexpr int RT = 16;    // tokens staged at a time

template <typename T, int KPT, int MODE>
__global__ void __launch_bounds__(256) k_recur_scan(const __grid_constant__ RecurP P) {
    constexpr int DP = 8 * KPT;
    extern __shared__ __align__(16) float sm[];
    float* sq = sm;
    float* sk = sq + RT * DP;
    float* sa = sk + RT * DP;
    float* sv = sa + (MODE == DEC_CONST ? 0 : MODE == DEC_HEAD ? RT : RT * DP);
    const int tid = threadIdx.x, g = tid & 7, cl = tid >> 3;
    const int h = blockIdx.y, col = blockIdx.x * 32 + cl;
    const bool col_ok = col < P.dvp;
    const int hq = h / P.per;
    const float decay = MODE == DEC_CONST ? P.dec.decay[h] : 0.0f;
    const float D = MODE == DEC_HEAD ? P.dec.D[h] : 0.0f;

    float s[KPT];
    float* Srow = P.S + ((long)h * P.dvp + (col_ok ? col : 0)) * P.dp;
#pragma unroll
    for (int i = 0; i < KPT / 4; i++) {
        const int c = i * 32 + g * 4;
        float4 x = make_float4(0, 0, 0, 0);
        if (c < P.dp) x = *(const float4*)(Srow + c);
        s[4 * i] = x.x; s[4 * i + 1] = x.y; s[4 * i + 2] = x.z; s[4 * i + 3] = x.w;
    }

    for (int t0 = 0; t0 < P.T; t0 += RT) {
        const int nt = min(RT, P.T - t0);
        for (int e = tid; e < nt * DP; e += 256) {
            const int t = e / DP, c = e - t * DP;
            const long r = (long)(t0 + t) * P.ld + (long)hq * P.dp + c;
            const bool ok = c < P.dp;
            sq[e] = ok ? to_f(((const T*)P.q)[r]) : 0.0f;
            sk[e] = ok ? to_f(((const T*)P.k)[r]) : 0.0f;
            if (MODE == DEC_HEAD) {
                sk[e] *= P.dec.hdt[(long)(t0 + t) * P.dec.ldh + h];
                if (c == 0) sa[t] = expf(P.dec.hla[(long)(t0 + t) * P.dec.ldh + h]);
            }
            if (MODE == DEC_LOG) sa[e] = ok ? expf(P.dec.la[(long)(t0 + t) * P.dec.ldla + (long)h * P.dp + c]) : 0.0f;
            if (MODE == DEC_LOWRANK) {
                float z = 0.0f;
                if (ok) {
                    const T* a2 = (const T*)P.dec.a2 + ((long)h * P.dp + c) * P.dec.lda2;
                    for (int j = 0; j < P.dec.rank; j++) z = fmaf(to_f(a2[j]), to_f(((const T*)P.dec.a1)[j]), z);
                    z = expf(logsigmoid_f(z + P.dec.bias[h * P.dp + c]) * P.dec.inv_tau);
                }
                sa[e] = z;
            }
        }
        for (int e = tid; e < nt * 32; e += 256) {
            const int t = e >> 5, c = blockIdx.x * 32 + (e & 31);
            sv[e] = c < P.dvp ? to_f(((const T*)P.v)[(long)(t0 + t) * P.ld + (long)h * P.dvp + c]) : 0.0f;
        }
        __syncthreads();
        for (int t = 0; t < nt; t++) {
            const float v = sv[t * 32 + cl];
            float o = 0.0f;
#pragma unroll
            for (int i = 0; i < KPT / 4; i++) {
                const int c = t * DP + i * 32 + g * 4;
                const float4 k = *(const float4*)(sk + c), q = *(const float4*)(sq + c);
                float4 a = make_float4(decay, decay, decay, decay);
                if (MODE == DEC_HEAD) a = make_float4(sa[t], sa[t], sa[t], sa[t]);
                else if (MODE != DEC_CONST) a = *(const float4*)(sa + c);
                s[4 * i] = fmaf(a.x, s[4 * i], k.x * v);
                s[4 * i + 1] = fmaf(a.y, s[4 * i + 1], k.y * v);
                s[4 * i + 2] = fmaf(a.z, s[4 * i + 2], k.z * v);
                s[4 * i + 3] = fmaf(a.w, s[4 * i + 3], k.w * v);
                o = fmaf(q.x, s[4 * i], fmaf(q.y, s[4 * i + 1], fmaf(q.z, s[4 * i + 2], fmaf(q.w, s[4 * i + 3], o))));
            }
            o += __shfl_xor_sync(0xffffffffu, o, 1);
            o += __shfl_xor_sync(0xffffffffu, o, 2);
            o += __shfl_xor_sync(0xffffffffu, o, 4);
            if (g == 0 && col_ok) P.o[(long)(t0 + t) * P.ldo + (long)h * P.dvp + col] = MODE == DEC_HEAD ? fmaf(D, v, o) : o;
        }
        __syncthreads();
    }
    if (col_ok) {
#pragma unroll
        for (int i = 0; i < KPT / 4; i++) {
            const int c = i * 32 + g * 4;
            if (c < P.dp) *(float4*)(Srow + c) = make_float4(s[4 * i], s[4 * i + 1], s[4 * i + 2], s[4 * i + 3]);
        }
    }
}

template <typename T, int KPT, int MODE>
static int launch_scan(const RecurP& P, cudaStream_t s) {
    const size_t smem = ((size_t)RT * 8 * KPT * (MODE == DEC_CONST || MODE == DEC_HEAD ? 2 : 3) + (size_t)RT * 33) * 4;
    static PerDeviceOnce once;
    if (once.first())
        LT_CUDA(cudaFuncSetAttribute(k_recur_scan<T, KPT, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    k_recur_scan<T, KPT, MODE><<<dim3((P.dvp + 31) / 32, P.H), 256, smem, s>>>(P);
    return check_launch("lt_dn_recurrence");
}
template <typename T, int KPT>
static int launch_mode(const RecurP& P, int mode, cudaStream_t s) {
    if (mode == DEC_CONST) return launch_scan<T, KPT, DEC_CONST>(P, s);
    if (mode == DEC_LOG) return launch_scan<T, KPT, DEC_LOG>(P, s);
    if (mode == DEC_HEAD) return launch_scan<T, KPT, DEC_HEAD>(P, s);
    return launch_scan<T, KPT, DEC_LOWRANK>(P, s);
}
template <typename T>
static int launch_size(const RecurP& P, int mode, cudaStream_t s) {
    if (P.dp <= 32) return launch_mode<T, 4>(P, mode, s);
    if (P.dp <= 64) return launch_mode<T, 8>(P, mode, s);
    if (P.dp <= 128) return launch_mode<T, 16>(P, mode, s);
    if (P.dp <= 256) return launch_mode<T, 32>(P, mode, s);
    return launch_mode<T, 64>(P, mode, s);
}

}  // namespace dn
}  // namespace lt

using namespace lt;
using namespace lt::dn;

extern "C" int lt_dn_recurrence(const void* q, const void* k, const void* v, int ld, float* S, float* o, int ldo, int f32, int T,
                                int H, int dp, int dvp, const lt_dn_decay* h_decay, void* stream) {
    LT_REQUIRE(q && k && v && S && o && h_decay, "lt_dn_recurrence: null pointer");
    LT_REQUIRE(T > 0 && H > 0 && dp > 0 && dvp > 0 && dp % 8 == 0 && dvp % 8 == 0, "lt_dn_recurrence: T=%d H=%d dp=%d dvp=%d", T, H, dp, dvp);
    LT_REQUIRE(dp <= 512, "lt_dn_recurrence: key size %d of a head is above 512", dp);
    LT_REQUIRE(aligned16(S), "lt_dn_recurrence: the state must be 16-byte aligned");
    RecurP P = {q, k, v, S, o, ld, ldo, T, H, dp, dvp, 1, *h_decay};
    int mode;
    if (h_decay->decay) mode = DEC_CONST;
    else if (h_decay->la) mode = DEC_LOG;
    else if (h_decay->hla) {
        mode = DEC_HEAD;
        LT_REQUIRE(h_decay->hdt && h_decay->D && h_decay->ldh >= H && h_decay->per > 0 && H % h_decay->per == 0,
                   "lt_dn_recurrence: step sizes, D, or %d heads in groups of %d", H, h_decay->per);
        P.per = h_decay->per;
    }
    else {
        mode = DEC_LOWRANK;
        LT_REQUIRE(T == 1 && h_decay->a1 && h_decay->a2 && h_decay->bias && h_decay->rank > 0,
                   "lt_dn_recurrence: the low-rank decay form takes one token (T=%d) and a1, a2, bias", T);
    }
    if (f32) return launch_size<float>(P, mode, (cudaStream_t)stream);
    return launch_size<bf16>(P, mode, (cudaStream_t)stream);
}
