// State-space mixer: what stands around its recurrence.  A causal convolution of a few taps per channel and silu ahead of it,
// step sizes softplus(dt + bias) and log decays A * step size; for one token the convolution and the recurrence in one launch.
#include "lt_dn_common.cuh"

namespace lt {
namespace dn {

template <typename T>
__device__ __forceinline__ float silu_t(float v) { return sizeof(T) == 2 ? silu_bf16(v) : v * sigmoid_f(v); }

// ---------------------------------------------------------------------------- rows of a portion

struct SsdRowsP {
    const void* u;
    const float* dt;
    void *ring, *out;
    float *hla, *hdt;
    int ld, lddt, ldo, T, pos0, C, nconv;
    lt_dn_ssd S;
};

constexpr int RUN = 8;      // tokens of a thread

// one 16-byte vector of the inputs at token t of the portion (t < 0: from the ring, zeros before the start)
template <typename T>
__device__ __forceinline__ void conv_input(const SsdRowsP& P, int t, int c, float (&f)[Vec<T>::N]) {
    const T* p = nullptr;
    if (t >= 0) {
        if (t < P.T) p = (const T*)P.u + (long)t * P.ld + c;
    } else if (P.pos0 + t >= 0) {
        p = (const T*)P.ring + (long)((P.pos0 + t) % P.S.taps) * P.C + c;
    }
    const uint4 v = p != nullptr ? *(const uint4*)p : make_uint4(0, 0, 0, 0);
    Vec<T>::unpack(v, f);
}

// TAPS > 0: taps and the sliding window in registers; 0: any number
template <typename T, int TAPS>
__global__ void __launch_bounds__(256) k_ssd_rows(const __grid_constant__ SsdRowsP P) {
    constexpr int N = Vec<T>::N;
    if ((int)blockIdx.x >= P.nconv) {
        const int H = P.S.H;
        const long i = (long)(blockIdx.x - P.nconv) * 256 + threadIdx.x;
        if (i >= (long)P.T * H) return;
        const int t = (int)(i / H), h = (int)(i - (long)t * H);
        const float d = softplus_f(P.dt[(long)t * P.lddt + h] + P.S.dt_bias[h]);
        P.hdt[i] = d;
        P.hla[i] = P.S.A[h] * d;
        return;
    }
    const int nc = P.C / N, runs = (P.T + RUN - 1) / RUN;
    const long i = (long)blockIdx.x * 256 + threadIdx.x;
    if (i >= (long)nc * runs) return;
    const int c = (int)(i % nc) * N, t0 = (int)(i / nc) * RUN;
    float b[N];
#pragma unroll
    for (int j = 0; j < N; j++) b[j] = P.S.conv_b[c + j];
    T* out = (T*)P.out + (long)t0 * P.ldo + c;
    auto store = [&](int t, float (&a)[N]) {
        T o[N];
#pragma unroll
        for (int j = 0; j < N; j++) o[j] = from_f<T>(silu_t<T>(a[j]));
        *(uint4*)(out + (long)t * P.ldo) = *(const uint4*)o;
    };
    if (TAPS > 0) {
        constexpr int K = TAPS > 0 ? TAPS : 1;
        float w[K][N], x[K][N];
#pragma unroll
        for (int k = 0; k < K; k++)
#pragma unroll
            for (int j = 0; j < N; j++) w[k][j] = P.S.conv[k * P.C + c + j];
#pragma unroll
        for (int k = 0; k < K - 1; k++) conv_input<T>(P, t0 - (K - 1) + k, c, x[k]);
#pragma unroll
        for (int t = 0; t < RUN; t++) {
            if (t0 + t >= P.T) break;
            conv_input<T>(P, t0 + t, c, x[K - 1]);
            float a[N];
#pragma unroll
            for (int j = 0; j < N; j++) {
                a[j] = b[j];
#pragma unroll
                for (int k = 0; k < K; k++) a[j] = fmaf(w[k][j], x[k][j], a[j]);
            }
            store(t, a);
#pragma unroll
            for (int k = 0; k < K - 1; k++)
#pragma unroll
                for (int j = 0; j < N; j++) x[k][j] = x[k + 1][j];
        }
    } else {
        const int taps = P.S.taps;
        for (int t = 0; t < RUN && t0 + t < P.T; t++) {
            float a[N];
#pragma unroll
            for (int j = 0; j < N; j++) a[j] = b[j];
            for (int k = 0; k < taps; k++) {
                float x[N];
                conv_input<T>(P, t0 + t - (taps - 1) + k, c, x);
#pragma unroll
                for (int j = 0; j < N; j++) a[j] = fmaf(P.S.conv[(long)k * P.C + c + j], x[j], a[j]);
            }
            store(t, a);
        }
    }
}

// the portion's last inputs into the ring (a launch of its own: the rows above read what this overwrites)
template <typename T>
__global__ void __launch_bounds__(256) k_ssd_keep(const __grid_constant__ SsdRowsP P) {
    constexpr int N = Vec<T>::N;
    const int nc = P.C / N, keep = min(P.T, P.S.taps);
    const int i = blockIdx.x * 256 + threadIdx.x;
    if (i >= nc * keep) return;
    const int t = P.T - keep + i / nc, c = (i % nc) * N;
    *(uint4*)((T*)P.ring + (long)((P.pos0 + t) % P.S.taps) * P.C + c) = *(const uint4*)((const T*)P.u + (long)t * P.ld + c);
}

template <typename T>
static int launch_rows(SsdRowsP& P, cudaStream_t s) {
    const int nc = P.C / Vec<T>::N;
    const long units = (long)nc * ((P.T + RUN - 1) / RUN);
    P.nconv = (int)((units + 255) / 256);
    const int grid = P.nconv + (int)(((long)P.T * P.S.H + 255) / 256);
    switch (P.S.taps) {
        case 2: k_ssd_rows<T, 2><<<grid, 256, 0, s>>>(P); break;
        case 3: k_ssd_rows<T, 3><<<grid, 256, 0, s>>>(P); break;
        case 4: k_ssd_rows<T, 4><<<grid, 256, 0, s>>>(P); break;
        default: k_ssd_rows<T, 0><<<grid, 256, 0, s>>>(P);
    }
    int rc = check_launch("lt_dn_ssd_rows");
    if (rc != LT_OK) return rc;
    const int keep = P.T < P.S.taps ? P.T : P.S.taps;
    k_ssd_keep<T><<<(nc * keep + 255) / 256, 256, 0, s>>>(P);
    return check_launch("lt_dn_ssd_rows (ring)");
}

// ---------------------------------------------------------------------------- one token

struct SsdStepP {
    const void* u;
    const float* dt;
    void* ring;
    float *state, *o;
    int *len, *ticket;
    int C;
    lt_dn_ssd S;
};

// CTA (x, h): 32 value columns of head h, eight lanes per column, dp / 8 key channels each in registers
template <typename T, int KPT>
__global__ void __launch_bounds__(256) k_ssd_step(const __grid_constant__ SsdStepP P) {
    constexpr int DP = 8 * KPT;
    __shared__ __align__(16) float sk[DP], sq[DP];
    __shared__ float sv[32];
    const lt_dn_ssd& S = P.S;
    const int tid = threadIdx.x, g = tid & 7, cl = tid >> 3;
    const int h = blockIdx.y, per = S.H / S.G, grp = h / per, col = blockIdx.x * 32 + cl;
    const bool col_ok = col < S.dvp;
    float s[KPT];
    float* row = P.state + ((long)h * S.dvp + (col_ok ? col : 0)) * S.dp;
#pragma unroll
    for (int i = 0; i < KPT / 4; i++) {
        const int c = i * 32 + g * 4;
        float4 x = make_float4(0, 0, 0, 0);
        if (c < S.dp) x = *(const float4*)(row + c);
        s[4 * i] = x.x; s[4 * i + 1] = x.y; s[4 * i + 2] = x.z; s[4 * i + 3] = x.w;
    }
    const int pos = *P.len, slot = pos % S.taps;
    const float dt = softplus_f(P.dt[h] + S.dt_bias[h]), a = expf(S.A[h] * dt), D = S.D[h];
    // channel c after convolution and silu; the new input goes to its slot of the ring, which no reader of this step needs
    auto channel = [&](int c, bool keep) {
        const T u = ((const T*)P.u)[c];
        float v = S.conv_b[c];
        int r = slot;
        for (int k = 0; k < S.taps - 1; k++) {       // positions pos - taps + 1 .. pos - 1
            r = r + 1 == S.taps ? 0 : r + 1;
            if (pos - (S.taps - 1) + k >= 0) v = fmaf(S.conv[(long)k * P.C + c], to_f(((const T*)P.ring)[(long)r * P.C + c]), v);
        }
        v = fmaf(S.conv[(long)(S.taps - 1) * P.C + c], to_f(u), v);
        if (keep) ((T*)P.ring)[(long)slot * P.C + c] = u;
        return to_f(from_f<T>(silu_t<T>(v)));
    };
    const bool first = blockIdx.x == 0 && h == grp * per;
    for (int e = tid; e < 2 * DP + 32; e += 256) {
        if (e < 2 * DP) {
            const int c = e < DP ? e : e - DP;
            float v = 0.0f;
            if (c < S.dp) v = channel(S.H * S.dvp + (e < DP ? 0 : S.G * S.dp) + grp * S.dp + c, first);
            if (e < DP) sk[c] = v * dt;
            else sq[c] = v;
        } else {
            const int c = blockIdx.x * 32 + e - 2 * DP;
            sv[e - 2 * DP] = c < S.dvp ? channel(h * S.dvp + c, true) : 0.0f;
        }
    }
    __syncthreads();
    const float v = sv[cl];
    float o = 0.0f;
#pragma unroll
    for (int i = 0; i < KPT / 4; i++) {
        const int c = i * 32 + g * 4;
        const float4 k = *(const float4*)(sk + c), q = *(const float4*)(sq + c);
        s[4 * i] = fmaf(a, s[4 * i], k.x * v);
        s[4 * i + 1] = fmaf(a, s[4 * i + 1], k.y * v);
        s[4 * i + 2] = fmaf(a, s[4 * i + 2], k.z * v);
        s[4 * i + 3] = fmaf(a, s[4 * i + 3], k.w * v);
        o = fmaf(q.x, s[4 * i], fmaf(q.y, s[4 * i + 1], fmaf(q.z, s[4 * i + 2], fmaf(q.w, s[4 * i + 3], o))));
        if (col_ok && c < S.dp) *(float4*)(row + c) = make_float4(s[4 * i], s[4 * i + 1], s[4 * i + 2], s[4 * i + 3]);
    }
    o += __shfl_xor_sync(0xffffffffu, o, 1);
    o += __shfl_xor_sync(0xffffffffu, o, 2);
    o += __shfl_xor_sync(0xffffffffu, o, 4);
    if (g == 0 && col_ok) P.o[(long)h * S.dvp + col] = fmaf(D, v, o);
    if (tid == 0) {      // past the barrier: every thread of this CTA has read the position
        if (atomicAdd(P.ticket, 1) == (int)(gridDim.x * gridDim.y) - 1) {
            *P.ticket = 0;
            *P.len = pos + 1;
        }
    }
}

template <typename T>
static int launch_ssd_step(const SsdStepP& P, cudaStream_t s) {
    const dim3 grid((P.S.dvp + 31) / 32, P.S.H);
    if (P.S.dp <= 32) k_ssd_step<T, 4><<<grid, 256, 0, s>>>(P);
    else if (P.S.dp <= 64) k_ssd_step<T, 8><<<grid, 256, 0, s>>>(P);
    else if (P.S.dp <= 128) k_ssd_step<T, 16><<<grid, 256, 0, s>>>(P);
    else if (P.S.dp <= 256) k_ssd_step<T, 32><<<grid, 256, 0, s>>>(P);
    else k_ssd_step<T, 64><<<grid, 256, 0, s>>>(P);
    return check_launch("lt_dn_ssd_step");
}

static const char* ssd_error(const lt_dn_ssd* S) {
    if (S == nullptr) return "null description";
    if (S->H <= 0 || S->G <= 0 || S->H % S->G || S->dp <= 0 || S->dvp <= 0 || S->taps <= 0) return "sizes";
    if (S->dp % 8 || S->dvp % 8) return "padded sizes must be multiples of 8";
    if (S->dp > 512) return "a state of more than 512 rows";
    if (!S->conv || !S->conv_b || !S->dt_bias || !S->A || !S->D) return "null constants";
    return nullptr;
}

}  // namespace dn
}  // namespace lt

using namespace lt;
using namespace lt::dn;

extern "C" int lt_dn_ssd_rows(const void* xbc, int ld, const float* dt, int lddt, void* ring, void* out, int ldo, float* hla, float* hdt,
                              int f32, int T, int pos0, const lt_dn_ssd* h_s, void* stream) {
    const char* bad = ssd_error(h_s);
    LT_REQUIRE(bad == nullptr, "lt_dn_ssd_rows: %s", bad);
    LT_REQUIRE(xbc && dt && ring && out && hla && hdt && T > 0 && pos0 >= 0, "lt_dn_ssd_rows: null pointer or T=%d pos0=%d", T, pos0);
    const int C = h_s->H * h_s->dvp + 2 * h_s->G * h_s->dp;
    LT_REQUIRE(ld % 8 == 0 && ld >= C && ldo % 8 == 0 && ldo >= C && lddt >= h_s->H, "lt_dn_ssd_rows: ld=%d ldo=%d lddt=%d for %d channels", ld, ldo, lddt, C);
    LT_REQUIRE(aligned16(xbc) && aligned16(ring) && aligned16(out), "lt_dn_ssd_rows: pointers must be 16-byte aligned");
    SsdRowsP P = {xbc, dt, ring, out, hla, hdt, ld, lddt, ldo, T, pos0, C, 0, *h_s};
    if (f32) return launch_rows<float>(P, (cudaStream_t)stream);
    return launch_rows<bf16>(P, (cudaStream_t)stream);
}

extern "C" int lt_dn_ssd_step(const void* xbc, const float* dt, void* ring, float* S, float* o, int f32, int* len, int* ticket,
                              const lt_dn_ssd* h_s, void* stream) {
    const char* bad = ssd_error(h_s);
    LT_REQUIRE(bad == nullptr, "lt_dn_ssd_step: %s", bad);
    LT_REQUIRE(xbc && dt && ring && S && o && len && ticket, "lt_dn_ssd_step: null pointer");
    LT_REQUIRE(aligned16(S), "lt_dn_ssd_step: the state must be 16-byte aligned");
    SsdStepP P = {xbc, dt, ring, S, o, len, ticket, h_s->H * h_s->dvp + 2 * h_s->G * h_s->dp, *h_s};
    if (f32) return launch_ssd_step<float>(P, (cudaStream_t)stream);
    return launch_ssd_step<bf16>(P, (cudaStream_t)stream);
}
