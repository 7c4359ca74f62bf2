// The state-space recurrence S <- a_t S + dt_t k_t x_t^T, o_t = S^T q_t + D x_t over a prompt portion in chunks of 64 tokens on
// the tensor cores (mma.sync m16n8k16, fp32 accumulation).  a_t and dt_t are numbers per head, q and k are shared by the heads
// of a group, so decays never have to be folded into q and k.  With b_t the sum of the chunk's log decays up to and
// including t:
//   k_ssd_states   a CTA owns a slice of one head's state and walks the chunks in order, the state in its accumulators:
//                  stores the state a chunk starts from, then S <- e^(b_end) S + sum_j (x_j dt_j e^(b_end - b_j)) k_j^T
//   k_ssd_out      every chunk at once; a CTA computes q_t . k_j once for its heads, then per head
//                  o_t = e^(b_t) S^T q_t + sum_(j <= t) (q_t . k_j) dt_j e^(b_t - b_j) x_j + D x_t
// q, k and x enter as the bf16 they are; what a decay has touched, and the state, as the sum of two bf16 (16 significant bits).
#include "lt_dn_chunk.cuh"
#include "lt_dn_mma.cuh"

namespace lt {
namespace dn {

constexpr int VT = 64;      // value columns of a tile
constexpr int VS = VT + 8;  // row stride of a value tile: an odd number of 16-byte units

// Stored states: quads of key channels as {hi, hi, lo, lo}, two bf16 each.  Quad 4 b + i of a row holds the channels 2 i,
// 2 i + 1, 2 i + 8, 2 i + 9 of the block of 16 channels b: what a lane of k_ssd_states has in its accumulators and a lane of
// k_ssd_out needs as an operand.

// x_t rows t0 .. t0 + 63, columns v0 .. v0 + 63 of head h, zeros outside
__device__ __forceinline__ void load_values(bf16* dst, const SsdChunkP& P, int h, int t0, int v0) {
    for (int e = threadIdx.x; e < CH * (VT / 8); e += 128) {
        const int t = e >> 3, c = (e & 7) * 8;
        const bool ok = t0 + t < P.T && v0 + c < P.dvp;
        cp16(dst + t * VS + c, P.v + (ok ? (long)(t0 + t) * P.ld + (long)h * P.dvp + v0 + c : 0), ok);
    }
}

// CS: key channels of a CTA
template <int CS>
struct SsdStates {
    static constexpr int KS = CS + 8, CW = CS / 2;      // row stride of a key tile, channels of a warp
    static constexpr int STAGES = 4;                    // chunks in flight
    static constexpr int STAGE = CH * (KS + VS) * 2 + 2 * CH * 4;
    static constexpr int SMEM = STAGES * STAGE;
};

template <int CS>
__global__ void __launch_bounds__(256) k_ssd_states(const __grid_constant__ SsdChunkP P) {
    using L = SsdStates<CS>;
    constexpr int KS = L::KS, CW = L::CW;
    extern __shared__ __align__(16) unsigned char smem[];      // per stage: keys, values, log decays, step sizes
    __shared__ __align__(16) float sw[8][CH];         // weights of the tokens, one copy per warp
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tg = lane & 3;
    const int c0 = blockIdx.x * CS, v0 = blockIdx.y * VT, h = blockIdx.z, hq = h / P.per, dk = (P.dp + 15) & ~15;
    const int vw = (warp & 3) * 16, cw = (warp >> 2) * CW, cb = c0 + cw;
    const int va = v0 + vw + g, vb = va + 8;

    // this thread's 16-byte units of the tiles: one column, every KR-th or 32nd row
    constexpr int KR = 256 / (CS / 8);
    const int kt = tid / (CS / 8), kc = (tid % (CS / 8)) * 8, vt = tid >> 3, vc = (tid & 7) * 8;
    const bool k_ok = c0 + kc < P.dp, v_ok = v0 + vc < P.dvp;
    const bf16* kp = P.k + (long)kt * P.ld + (long)hq * P.dp + c0 + kc;
    const bf16* vp = P.v + (long)vt * P.ld + (long)h * P.dvp + v0 + vc;
    const long kstep = (long)KR * P.ld, vstep = 32L * P.ld, cstep = (long)CH * P.ld;
    const float* np = tid < CH ? P.hla : P.hdt;
    auto load = [&](int chunk) {      // of the chunks in order; an empty group past the last
        if (chunk >= P.nchunk) {
            asm volatile("cp.async.commit_group;" ::: "memory");
            return;
        }
        bf16* sk = (bf16*)(smem + (chunk % L::STAGES) * L::STAGE);
        bf16* sv = sk + CH * KS;
        float* sl = (float*)(sv + CH * VS);
        const int rows = P.T - chunk * CH;
#pragma unroll
        for (int i = 0; i < CH / KR; i++) {
            const bool ok = k_ok && kt + i * KR < rows;
            cp16(&sk[(kt + i * KR) * KS + kc], ok ? kp + i * kstep : P.k, ok);
        }
#pragma unroll
        for (int i = 0; i < CH / 32; i++) {
            const bool ok = v_ok && vt + i * 32 < rows;
            cp16(&sv[(vt + i * 32) * VS + vc], ok ? vp + i * vstep : P.v, ok);
        }
        if (tid < 2 * CH) {
            const bool ok = (tid & 63) < rows;
            cp4(&sl[tid], ok ? np + (long)(chunk * CH + (tid & 63)) * P.ldh + h : np, ok);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        kp += cstep;
        vp += cstep;
    };
    float acc[CW / 8][4];               // S[va or vb][cb + 8 i + 2 tg + (0, 1)]
#pragma unroll
    for (int i = 0; i < CW / 8; i++) {
        const int c = cb + i * 8 + tg * 2;
        float2 a = make_float2(0, 0), b = a;
        if (c < P.dp && va < P.dvp) a = *(const float2*)(P.S + ((long)h * P.dvp + va) * P.dp + c);
        if (c < P.dp && vb < P.dvp) b = *(const float2*)(P.S + ((long)h * P.dvp + vb) * P.dp + c);
        acc[i][0] = a.x; acc[i][1] = a.y; acc[i][2] = b.x; acc[i][3] = b.y;
    }
#pragma unroll
    for (int i = 0; i < L::STAGES - 1; i++) load(i);
    for (int chunk = 0; chunk < P.nchunk; chunk++) {
        asm volatile("cp.async.wait_group %0;" ::"n"(L::STAGES - 2) : "memory");
        __syncthreads();                // the chunk is there, and nobody reads the stage of the one before
        load(chunk + L::STAGES - 1);
        const bf16* sk = (const bf16*)(smem + (chunk % L::STAGES) * L::STAGE);
        const bf16* sv = sk + CH * KS;
        const float* sl = (const float*)(sv + CH * VS);
        // the state the chunk starts from
        uint4* w = (uint4*)P.ws + (((long)chunk * P.H + h) * P.dvp) * (dk >> 2) + tg;
#pragma unroll
        for (int i = 0; i < CW / 8; i += 2) {
            const int c = cb + i * 8;
            if (c >= dk) break;
            unsigned h0, h1, l0, l1;
            if (va < P.dvp) {
                split2(acc[i][0], acc[i][1], h0, l0);
                split2(acc[i + 1][0], acc[i + 1][1], h1, l1);
                w[(long)va * (dk >> 2) + (c >> 2)] = make_uint4(h0, h1, l0, l1);
            }
            if (vb < P.dvp) {
                split2(acc[i][2], acc[i][3], h0, l0);
                split2(acc[i + 1][2], acc[i + 1][3], h1, l1);
                w[(long)vb * (dk >> 2) + (c >> 2)] = make_uint4(h0, h1, l0, l1);
            }
        }
        // weights dt_j e^(b_end - b_j): sums of the log decays behind j, two tokens per lane
        const float la0 = sl[2 * lane] * LOG2E, la1 = sl[2 * lane + 1] * LOG2E;
        float p = la0 + la1;
#pragma unroll
        for (int s = 1; s < 32; s <<= 1) {
            const float x = __shfl_down_sync(0xffffffffu, p, s);
            if (lane + s < 32) p += x;
        }
        float behind = __shfl_down_sync(0xffffffffu, p, 1);
        if (lane == 31) behind = 0.0f;
        *(float2*)&sw[warp][2 * lane] = make_float2(exp2f(behind + la1) * sl[CH + 2 * lane], exp2f(behind) * sl[CH + 2 * lane + 1]);
        const float a = exp2f(__shfl_sync(0xffffffffu, p, 0));
#pragma unroll
        for (int i = 0; i < CW / 8; i++) {
            acc[i][0] *= a; acc[i][1] *= a; acc[i][2] *= a; acc[i][3] *= a;
        }
        __syncwarp();
#pragma unroll
        for (int kk = 0; kk < CH / 16; kk++) {
            unsigned x[4], hi[4], lo[4];
            ldsm4t(x, &sv[(kk * 16 + (lane >> 4) * 8 + (lane & 7)) * VS + vw + ((lane >> 3) & 1) * 8]);
            const float2 w0 = *(const float2*)&sw[warp][kk * 16 + 2 * tg], w1 = *(const float2*)&sw[warp][kk * 16 + 8 + 2 * tg];
            split2(lo_f(x[0]) * w0.x, hi_f(x[0]) * w0.y, hi[0], lo[0]);
            split2(lo_f(x[1]) * w0.x, hi_f(x[1]) * w0.y, hi[1], lo[1]);
            split2(lo_f(x[2]) * w1.x, hi_f(x[2]) * w1.y, hi[2], lo[2]);
            split2(lo_f(x[3]) * w1.x, hi_f(x[3]) * w1.y, hi[3], lo[3]);
#pragma unroll
            for (int i = 0; i < CW / 8; i += 2) {
                unsigned r[4];
                ldsm4t(r, &sk[(kk * 16 + (lane & 15)) * KS + cw + i * 8 + (lane >> 4) * 8]);
                mma16816(acc[i], hi, r[0], r[1]);
                mma16816(acc[i + 1], hi, r[2], r[3]);
                mma16816(acc[i], lo, r[0], r[1]);
                mma16816(acc[i + 1], lo, r[2], r[3]);
            }
        }
        __syncwarp();                   // sw is written again
    }
#pragma unroll
    for (int i = 0; i < CW / 8; i++) {
        const int c = cb + i * 8 + tg * 2;
        if (c >= P.dp) break;
        if (va < P.dvp) *(float2*)(P.S + ((long)h * P.dvp + va) * P.dp + c) = make_float2(acc[i][0], acc[i][1]);
        if (vb < P.dvp) *(float2*)(P.S + ((long)h * P.dvp + vb) * P.dp + c) = make_float2(acc[i][2], acc[i][3]);
    }
}

// NK: blocks of 16 key channels at most; a warp owns 16 tokens
template <int NK>
struct SsdOut {
    static constexpr int QS = NK * 16 + 8;       // row strides: q and k in bf16, states in 32-bit words (16 banks apart)
    static constexpr int BS = NK * 16 + 16;
    static constexpr int QK = 2 * CH * QS * 2, SV = VT * BS * 4 + CH * VS * 2;
    static constexpr int SMEM = QK > SV ? QK : SV;
    static constexpr int CTAS = NK <= 8 ? 4 : 2;      // of an SM
};

template <int NK>
__global__ void __launch_bounds__(128, SsdOut<NK>::CTAS) k_ssd_out(const __grid_constant__ SsdChunkP P) {
    using L = SsdOut<NK>;
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ __align__(16) double sd[CH];      // running sums of the log decays (double: differences are exact)
    __shared__ float sdt[CH];
    bf16* sq = (bf16*)smem;
    bf16* sk = sq + CH * L::QS;
    unsigned* sS = (unsigned*)smem;              // over q and k, once they are used
    bf16* sv = (bf16*)(sS + VT * L::BS);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tg = lane & 3;
    const int chunk = blockIdx.x, t0 = chunk * CH, nk = (P.dp + 15) >> 4, dk = nk * 16;
    const int grp = blockIdx.y / P.nb, hb = blockIdx.y - grp * P.nb;
    const int h0 = grp * P.per + hb * P.hpc, h1 = min(h0 + P.hpc, (grp + 1) * P.per);

    for (int e = tid; e < CH * 2 * nk; e += 128) {
        const int t = e / (2 * nk), c = (e - t * 2 * nk) * 8;
        const bool ok = t0 + t < P.T && c < P.dp;
        const long off = ok ? (long)(t0 + t) * P.ld + (long)grp * P.dp + c : 0;
        cp16(sq + t * L::QS + c, P.q + off, ok);
        cp16(sk + t * L::QS + c, P.k + off, ok);
    }
    asm volatile("cp.async.commit_group;\n\tcp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    unsigned qf[NK][4];
    float s[8][4];                               // q_t . k_j: t = 16 warp + g (+ 8), j = 8 n + 2 tg (+ 1), up to the diagonal
#pragma unroll
    for (int n = 0; n < 8; n++) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.0f;
#pragma unroll
    for (int kk = 0; kk < NK; kk++) {
        if (kk >= nk) break;
        ldsm4(qf[kk], sq + (warp * 16 + (lane & 15)) * L::QS + kk * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int n = 0; n < 8; n += 2) {
            if (n > 2 * warp) break;
            unsigned r[4];
            ldsm4(r, sk + (n * 8 + (lane & 7) + ((lane >> 4) << 3)) * L::QS + kk * 16 + ((lane >> 3) & 1) * 8);
            mma16816(s[n], qf[kk], r[0], r[1]);
            mma16816(s[n + 1], qf[kk], r[2], r[3]);
        }
    }
    const int ta = warp * 16 + g, tb = ta + 8;
    for (int h = h0; h < h1; h++) {
        for (int v0 = 0; v0 < P.dvp; v0 += VT) {
            __syncthreads();
            const uint4* src = (const uint4*)P.ws + (((long)chunk * P.H + h) * P.dvp + v0) * (dk >> 2);
            const int nu = dk >> 2;
            for (int e = tid; e < VT * nu; e += 128) {
                const int v = e / nu, c = e - v * nu;
                const bool ok = v0 + v < P.dvp;
                cp16(sS + v * L::BS + c * 4, src + (ok ? (long)v * nu + c : 0), ok);
            }
            load_values(sv, P, h, t0, v0);
            asm volatile("cp.async.commit_group;" ::: "memory");
            if (v0 == 0 && warp == 0) {
                const int t = t0 + 2 * lane;
                const float l0 = t < P.T ? P.hla[(long)t * P.ldh + h] * LOG2E : 0.0f;
                const float l1 = t + 1 < P.T ? P.hla[(long)(t + 1) * P.ldh + h] * LOG2E : 0.0f;
                sdt[2 * lane] = t < P.T ? P.hdt[(long)t * P.ldh + h] : 0.0f;
                sdt[2 * lane + 1] = t + 1 < P.T ? P.hdt[(long)(t + 1) * P.ldh + h] : 0.0f;
                double p = (double)l0 + (double)l1;
#pragma unroll
                for (int i = 1; i < 32; i <<= 1) {
                    const double x = __shfl_up_sync(0xffffffffu, p, i);
                    if (lane >= i) p += x;
                }
                double before = __shfl_up_sync(0xffffffffu, p, 1);
                if (lane == 0) before = 0.0;
                sd[2 * lane] = before + (double)l0;
                sd[2 * lane + 1] = p;
            }
            asm volatile("cp.async.wait_group 0;" ::: "memory");
            __syncthreads();

            const double da = sd[ta], db = sd[tb];
            const float fa = exp2f((float)da), fb = exp2f((float)db);
            float acc[8][4];
#pragma unroll
            for (int n = 0; n < 8; n++) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.0f;
#pragma unroll
            for (int kk = 0; kk < NK; kk++) {
                if (kk >= nk) break;
#pragma unroll
                for (int n = 0; n < 8; n++) {
                    const uint4 r = *(const uint4*)(sS + (n * 8 + g) * L::BS + kk * 16 + tg * 4);
                    mma16816(acc[n], qf[kk], r.x, r.y);
                    mma16816(acc[n], qf[kk], r.z, r.w);
                }
            }
#pragma unroll
            for (int n = 0; n < 8; n++) {
                acc[n][0] *= fa; acc[n][1] *= fa; acc[n][2] *= fb; acc[n][3] *= fb;
            }
#pragma unroll
            for (int kk = 0; kk < CH / 16; kk++) {
                if (kk > warp) break;
                unsigned hi[4], lo[4];
#pragma unroll
                for (int i = 0; i < 2; i++) {
                    const int n = 2 * kk + i, j = n * 8 + 2 * tg;
                    const double2 dj = *(const double2*)&sd[j];
                    const float2 dt = *(const float2*)&sdt[j];
                    float x[4] = {s[n][0] * dt.x, s[n][1] * dt.y, s[n][2] * dt.x, s[n][3] * dt.y};
                    x[0] = j <= ta ? x[0] * exp2f((float)(da - dj.x)) : 0.0f;
                    x[1] = j + 1 <= ta ? x[1] * exp2f((float)(da - dj.y)) : 0.0f;
                    x[2] = j <= tb ? x[2] * exp2f((float)(db - dj.x)) : 0.0f;
                    x[3] = j + 1 <= tb ? x[3] * exp2f((float)(db - dj.y)) : 0.0f;
                    split2(x[0], x[1], hi[2 * i], lo[2 * i]);
                    split2(x[2], x[3], hi[2 * i + 1], lo[2 * i + 1]);
                }
#pragma unroll
                for (int n = 0; n < 8; n += 2) {
                    unsigned r[4];
                    ldsm4t(r, sv + (kk * 16 + (lane & 15)) * VS + n * 8 + (lane >> 4) * 8);
                    mma16816(acc[n], hi, r[0], r[1]);
                    mma16816(acc[n + 1], hi, r[2], r[3]);
                    mma16816(acc[n], lo, r[0], r[1]);
                    mma16816(acc[n + 1], lo, r[2], r[3]);
                }
            }
            const float D = P.D[h];
#pragma unroll
            for (int r = 0; r < 2; r++) {
                const int t = ta + r * 8;
                if (t0 + t >= P.T) continue;
                float* o = P.o + (long)(t0 + t) * P.ldo + (long)h * P.dvp + v0;
#pragma unroll
                for (int n = 0; n < 8; n++) {
                    const int v = n * 8 + 2 * tg;
                    if (v0 + v >= P.dvp) break;
                    const unsigned x = *(const unsigned*)(sv + t * VS + v);
                    *(float2*)(o + v) = make_float2(fmaf(D, lo_f(x), acc[n][2 * r]), fmaf(D, hi_f(x), acc[n][2 * r + 1]));
                }
            }
        }
    }
}

template <int NK>
static int launch_out(SsdChunkP P, cudaStream_t s) {
    static PerDeviceOnce once;
    if (once.first())
        LT_CUDA(cudaFuncSetAttribute(k_ssd_out<NK>, cudaFuncAttributeMaxDynamicSharedMemorySize, SsdOut<NK>::SMEM));
    // heads of a CTA: q . k is computed once for them, but the GPU should be filled in whole waves
    float best = 0.0f;
    for (int n = 1; n <= 8 && n <= P.per; n++) {
        const int nb = (P.per + n - 1) / n;
        const long ctas = (long)P.nchunk * (P.H / P.per) * nb, slots = (long)SsdOut<NK>::CTAS * sm_count();
        const float cost = (float)((ctas + slots - 1) / slots) * (n + 0.7f);
        if (n == 1 || cost < best) {
            best = cost;
            P.hpc = n;
            P.nb = nb;
        }
    }
    k_ssd_out<NK><<<dim3(P.nchunk, P.H / P.per * P.nb), 128, SsdOut<NK>::SMEM, s>>>(P);
    return check_launch("lt_dn_recurrence_chunked (state-space outputs)");
}

int launch_ssd_chunked(const SsdChunkP& P, cudaStream_t s) {
    const int nv = (P.dvp + VT - 1) / VT;
    static PerDeviceOnce once;
    if (once.first()) {
        LT_CUDA(cudaFuncSetAttribute(k_ssd_states<64>, cudaFuncAttributeMaxDynamicSharedMemorySize, SsdStates<64>::SMEM));
        LT_CUDA(cudaFuncSetAttribute(k_ssd_states<32>, cudaFuncAttributeMaxDynamicSharedMemorySize, SsdStates<32>::SMEM));
    }
    if ((long)P.H * nv * ((P.dp + 63) / 64) >= 100)
        k_ssd_states<64><<<dim3((P.dp + 63) / 64, nv, P.H), 256, SsdStates<64>::SMEM, s>>>(P);
    else
        k_ssd_states<32><<<dim3((P.dp + 31) / 32, nv, P.H), 256, SsdStates<32>::SMEM, s>>>(P);
    const int rc = check_launch("lt_dn_recurrence_chunked (state-space states)");
    if (rc != LT_OK) return rc;
    if (P.dp <= 64) return launch_out<4>(P, s);
    if (P.dp <= 128) return launch_out<8>(P, s);
    return launch_out<16>(P, s);
}

}  // namespace dn
}  // namespace lt
