// The recurrence S <- diag(a_t) S + k_t v_t^T, o_t = S^T q_t over a prompt portion, in chunks of 64 tokens on the tensor
// cores (mma.sync m16n8k16, fp32 accumulation).  With b_t the sum of the log decays of the chunk up to and including t:
//     dS        = sum_j (k_j e^(b_end - b_j)) v_j^T                            k_chunk_state, every chunk at once
//     S_next    = e^(b_end) S + dS                                            k_chunk_scan, element by element
//     o_t       = (q_t e^(b_t))^T S + sum_(j <= t) (q_t . k_j e^(b_t - b_j)) v_j   k_chunk_out, every chunk at once
// q, k and v are bf16 as they are; whatever a decay has touched, the state and the weights of the last sum enter their
// products as a sum of two bf16 (16 significant bits).  No exponential grows: the weights are formed in blocks of 16
// tokens, decays measured from the start of the query's block, (q_t e^(b_t - r)) . (k_j e^(r - b_j)); inside the block
// the second exponent is positive, and where it could leave a safe range the block's weights are summed pair by pair.
#include "lt_dn_chunk.cuh"
#include "lt_dn_mma.cuh"

namespace lt {
namespace dn {

constexpr float SAFE_EXP = 86.0f;              // of 2 (e^60)

struct ChunkP {
    const bf16 *q, *k, *v;
    float *S, *o, *ws, *dend;     // ws [chunk][H][dvp][dp]; dend [chunk][H][dp] (decay of a whole chunk)
    int ld, ldo, T, H, dp, dvp, nchunk;
    const float* decay;
    const float* la;
    int ldla;
};

// rows [t0, t0 + 64) x n columns of a bf16 matrix into shared memory, zero rows past T
__device__ __forceinline__ void load_tile(bf16* dst, int stride, const bf16* src, int ld, int t0, int T, int n) {
    const int nu = n >> 3;
    for (int e = threadIdx.x; e < CH * nu; e += blockDim.x) {
        const int t = e / nu, c = e - t * nu;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (t0 + t < T) v = *(const uint4*)(src + (long)(t0 + t) * ld + c * 8);
        *(uint4*)(dst + t * stride + c * 8) = v;
    }
}
__device__ __forceinline__ void load_logs(float* dst, int stride, const float* la, int ldla, int t0, int T, int n) {
    const int nu = n >> 2;
    for (int e = threadIdx.x; e < CH * nu; e += blockDim.x) {
        const int t = e / nu, c = e - t * nu;
        float4 v = make_float4(0, 0, 0, 0);
        if (t0 + t < T) v = *(const float4*)(la + (long)(t0 + t) * ldla + c * 4);
        v.x *= LOG2E; v.y *= LOG2E; v.z *= LOG2E; v.w *= LOG2E;
        *(float4*)(dst + t * stride + c * 4) = v;
    }
}

// ---------------------------------------------------------------------------- dS of every chunk

template <bool LOG>
__global__ void __launch_bounds__(256) k_chunk_state(const __grid_constant__ ChunkP P) {
    extern __shared__ __align__(16) unsigned char smem[];
    const int ks = P.dp + 8, vs = P.dvp + 8;      // an odd number of 16-byte units
    bf16* sh = (bf16*)smem;
    bf16* sl = sh + CH * ks;
    bf16* sv = sl + CH * ks;
    float* sla = (float*)(sv + CH * vs);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int chunk = blockIdx.x, h = blockIdx.y, t0 = chunk * CH, n = min(CH, P.T - t0);

    load_tile(sh, ks, P.k + (long)h * P.dp, P.ld, t0, P.T, P.dp);
    load_tile(sv, vs, P.v + (long)h * P.dvp, P.ld, t0, P.T, P.dvp);
    if (LOG) load_logs(sla, P.dp, P.la + (long)h * P.dp, P.ldla, t0, P.T, P.dp);
    __syncthreads();
    // k_j e^(b_end - b_j) as two bf16, in place
    if (LOG) {
        for (int e = tid; e < 4 * P.dp; e += 256) {
            const int seg = e / P.dp, c = e - seg * P.dp;
            float s = 0.0f;
            for (int j = CH - 1; j >= (seg + 1) * 16; j--) s += sla[j * P.dp + c];
            for (int j = seg * 16 + 15; j >= seg * 16; j--) {
                const float x = to_f(sh[j * ks + c]) * exp2f(s);
                const bf16 hi = from_f<bf16>(x);
                sh[j * ks + c] = hi;
                sl[j * ks + c] = from_f<bf16>(x - to_f(hi));
                s += sla[j * P.dp + c];
            }
            if (seg == 0) P.dend[((long)chunk * P.H + h) * P.dp + c] = exp2f(s);
        }
    } else {
        const float lam = P.decay[h];
        float* pw = sla;
        if (tid < CH) pw[tid] = tid < n ? powf(lam, (float)(n - 1 - tid)) : 0.0f;
        __syncthreads();
        for (int e = tid; e < CH * P.dp; e += 256) {
            const int j = e / P.dp, c = e - j * P.dp;
            const float x = to_f(sh[j * ks + c]) * pw[j];
            const bf16 hi = from_f<bf16>(x);
            sh[j * ks + c] = hi;
            sl[j * ks + c] = from_f<bf16>(x - to_f(hi));
        }
    }
    __syncthreads();
    // dS[v][c]: 16 value rows x 64 key columns at a time
    const int nv = (P.dvp + 15) >> 4, nc = (P.dp + 63) >> 6;
    float* out = P.ws + ((long)chunk * P.H + h) * P.dvp * P.dp;
    for (int it = warp; it < nv * nc; it += 8) {
        const int m0 = (it % nv) * 16, c0 = (it / nv) * 64;
        float acc[8][4];
#pragma unroll
        for (int i = 0; i < 8; i++) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.0f;
#pragma unroll
        for (int kk = 0; kk < CH / 16; kk++) {
            unsigned a[4];     // value columns past dvp fall into the row padding (8 elements), never stored
            ldsm4t(a, sv + (kk * 16 + (lane >> 4) * 8 + (lane & 7)) * vs + m0 + ((lane >> 3) & 1) * 8);
#pragma unroll
            for (int i = 0; i < 8; i += 2) {
                const int c = c0 + i * 8;
                if (c >= P.dp) break;
                unsigned r[4];
                const int off = (kk * 16 + (lane & 15)) * ks + c + (lane >> 4) * 8;
                ldsm4t(r, sh + off);
                mma16816(acc[i], a, r[0], r[1]);
                mma16816(acc[i + 1], a, r[2], r[3]);
                ldsm4t(r, sl + off);
                mma16816(acc[i], a, r[0], r[1]);
                mma16816(acc[i + 1], a, r[2], r[3]);
            }
        }
#pragma unroll
        for (int i = 0; i < 8; i++) {
            const int c = c0 + i * 8 + (lane & 3) * 2, v = m0 + (lane >> 2);
            if (c < P.dp) {
                if (v < P.dvp) *(float2*)(out + (long)v * P.dp + c) = make_float2(acc[i][0], acc[i][1]);
                if (v + 8 < P.dvp) *(float2*)(out + (long)(v + 8) * P.dp + c) = make_float2(acc[i][2], acc[i][3]);
            }
        }
    }
}

// ---------------------------------------------------------------------------- states between chunks

// Replaces dS of each chunk by the state the chunk starts from, four channels at a time as {4 x bf16 hi, 4 x bf16 lo}.
template <bool LOG>
__global__ void __launch_bounds__(256) k_chunk_scan(const __grid_constant__ ChunkP P) {
    const int nq = P.dp >> 2;
    const long i = (long)blockIdx.x * 256 + threadIdx.x, per = (long)P.H * P.dvp * nq;
    if (i >= per) return;
    const int cq = (int)(i % nq), h = (int)(i / nq / P.dvp);
    float4* S = (float4*)P.S + i;
    float4* w = (float4*)P.ws + i;
    float4 s = *S;
    float full = 0.0f, tail = 0.0f;
    if (!LOG) {
        full = powf(P.decay[h], (float)CH);
        tail = powf(P.decay[h], (float)(P.T - (P.nchunk - 1) * CH));
    }
    float4 nxt = w[0];
    for (int c = 0; c < P.nchunk; c++) {
        const float4 d = nxt;
        if (c + 1 < P.nchunk) nxt = w[(long)(c + 1) * per];
        unsigned h0, l0, h1, l1;
        split2(s.x, s.y, h0, l0);
        split2(s.z, s.w, h1, l1);
        *(uint4*)(w + (long)c * per) = make_uint4(h0, h1, l0, l1);
        float4 a;
        if (LOG) a = *(const float4*)(P.dend + ((long)c * P.H + h) * P.dp + cq * 4);
        else {
            const float f = c + 1 < P.nchunk ? full : tail;
            a = make_float4(f, f, f, f);
        }
        s.x = fmaf(a.x, s.x, d.x); s.y = fmaf(a.y, s.y, d.y);
        s.z = fmaf(a.z, s.z, d.z); s.w = fmaf(a.w, s.w, d.w);
    }
    *S = s;
}

// ---------------------------------------------------------------------------- outputs of every chunk

// Operand fragments hold channels 4g .. 4g+3 of every 16 in lane group g = lane & 3 (the contraction index may be
// permuted as long as both operands agree), so a lane reads four neighbouring channels at once.
struct Quad {
    float x[4];
};
__device__ __forceinline__ Quad load_quad(const bf16* p) {
    const uint2 r = *(const uint2*)p;
    Quad q;
    q.x[0] = lo_f(r.x); q.x[1] = hi_f(r.x); q.x[2] = lo_f(r.y); q.x[3] = hi_f(r.y);
    return q;
}

template <bool LOG>
__global__ void __launch_bounds__(256, 2) k_chunk_out(const __grid_constant__ ChunkP P) {
    extern __shared__ __align__(16) unsigned char smem[];
    const int qs = ((P.dp + 63) & ~63) + 16;       // bf16 row stride: rows 8 banks apart for 8-byte reads
    const int bs = ((P.dp + 31) & ~31) + 16;       // fp32 row stride: rows 16 banks apart for 16-byte reads
    const int vs = P.dvp + 8;
    constexpr int as = CH + 8;
    bf16* sq = (bf16*)smem;
    bf16* sk = sq + CH * qs;
    bf16* sv = sk + CH * qs;
    bf16* sAh = sv + CH * vs;
    bf16* sAl = sAh + CH * as;
    // LOG: sums of the log decays per channel, inside each block of 16 tokens (so that a difference inside a block does
    // not inherit the rounding of what came before), then sp[0..3]: what the blocks before block I add up to.
    // Else: powers of the head's decay.
    float* sb = (float*)(sAl + CH * as);
    float* sp = sb + CH * bs;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tg = lane & 3;
    const int chunk = blockIdx.x, h = blockIdx.y, t0 = chunk * CH;
    const int dk = (P.dp + 15) & ~15;              // contraction length; rows are zero past dp

    load_tile(sq, qs, P.q + (long)h * P.dp, P.ld, t0, P.T, P.dp);
    load_tile(sk, qs, P.k + (long)h * P.dp, P.ld, t0, P.T, P.dp);
    load_tile(sv, vs, P.v + (long)h * P.dvp, P.ld, t0, P.T, P.dvp);
    for (int e = tid; e < CH; e += 256) {
        *(uint4*)(sq + e * qs + P.dp) = make_uint4(0, 0, 0, 0);
        *(uint4*)(sk + e * qs + P.dp) = make_uint4(0, 0, 0, 0);
        *(uint4*)(sv + e * vs + P.dvp) = make_uint4(0, 0, 0, 0);
    }
    if (LOG) {
        load_logs(sb, bs, P.la + (long)h * P.dp, P.ldla, t0, P.T, P.dp);
        for (int e = tid; e < CH * 8; e += 256) sb[(e >> 3) * bs + P.dp + (e & 7)] = 0.0f;
        __syncthreads();
        for (int e = tid; e < 4 * (P.dp + 8); e += 256) {
            const int seg = e / (P.dp + 8), c = e - seg * (P.dp + 8);
            float s = 0.0f;
            for (int j = seg * 16; j < seg * 16 + 16; j++) {
                s += sb[j * bs + c];
                sb[j * bs + c] = s;
            }
        }
        __syncthreads();
        for (int c = tid; c < P.dp + 8; c += 256) {
            float s = 0.0f;
            for (int I = 0; I < 4; I++) {
                sp[I * bs + c] = s;
                s += sb[(I * 16 + 15) * bs + c];
            }
        }
    } else if (tid <= CH) {
        sb[tid] = powf(P.decay[h], (float)tid);
    }
    __syncthreads();

    // ---- weights A[t][j], j <= t: half blocks of 16 queries x 8 keys, I = query block, J = key block
    for (int it = warp; it < 20; it += 8) {
        const int half = it & 1, bl = it >> 1;
        const int I = bl == 0 ? 0 : (bl < 3 ? 1 : (bl < 6 ? 2 : 3)), J = bl - I * (I + 1) / 2;
        const int tq = I * 16 + g, tk = J * 16 + half * 8 + g;
        float acc[4] = {0.0f, 0.0f, 0.0f, 0.0f};
        bool direct = false;
        if (LOG && I == J) {      // largest exponent of k e^(r - b_j) in the block
            float mx = 0.0f;
            for (int c = lane; c < P.dp; c += 32)
                mx = fmaxf(mx, -sb[(I * 16 + 15) * bs + c]);
            direct = warp_max(mx) > SAFE_EXP;
        }
        if (!direct) {
            for (int kk = 0; kk < dk; kk += 16) {
                const int c = kk + tg * 4;
                Quad qa = load_quad(sq + tq * qs + c), qb = load_quad(sq + (tq + 8) * qs + c), kq = load_quad(sk + tk * qs + c);
                if (LOG) {
                    // query: from the start of its block; key: up to there (block J's rest, the blocks between)
                    const float4 ba = *(const float4*)(sb + tq * bs + c), bb = *(const float4*)(sb + (tq + 8) * bs + c);
                    const float4 bk = *(const float4*)(sb + tk * bs + c);
                    float4 r = make_float4(0, 0, 0, 0);
                    if (I > J) r = *(const float4*)(sb + (J * 16 + 15) * bs + c);
                    float rk[4] = {r.x - bk.x, r.y - bk.y, r.z - bk.z, r.w - bk.w};
                    for (int M = J + 1; M < I; M++) {
                        const float4 t = *(const float4*)(sb + (M * 16 + 15) * bs + c);
                        rk[0] += t.x; rk[1] += t.y; rk[2] += t.z; rk[3] += t.w;
                    }
                    const float ra[4] = {ba.x, ba.y, ba.z, ba.w};
                    const float rb[4] = {bb.x, bb.y, bb.z, bb.w};
#pragma unroll
                    for (int i = 0; i < 4; i++) {
                        qa.x[i] *= exp2f(ra[i]);
                        qb.x[i] *= exp2f(rb[i]);
                        kq.x[i] *= exp2f(rk[i]);
                    }
                    unsigned ah[4], al[4], bh[2], bl2[2];
                    split2(qa.x[0], qa.x[1], ah[0], al[0]);
                    split2(qb.x[0], qb.x[1], ah[1], al[1]);
                    split2(qa.x[2], qa.x[3], ah[2], al[2]);
                    split2(qb.x[2], qb.x[3], ah[3], al[3]);
                    split2(kq.x[0], kq.x[1], bh[0], bl2[0]);
                    split2(kq.x[2], kq.x[3], bh[1], bl2[1]);
                    mma16816(acc, ah, bh[0], bh[1]);
                    mma16816(acc, ah, bl2[0], bl2[1]);
                    mma16816(acc, al, bh[0], bh[1]);
                } else {
                    const uint2 ua = *(const uint2*)(sq + tq * qs + c), ub = *(const uint2*)(sq + (tq + 8) * qs + c);
                    const uint2 uk = *(const uint2*)(sk + tk * qs + c);
                    const unsigned a[4] = {ua.x, ub.x, ua.y, ub.y};
                    mma16816(acc, a, uk.x, uk.y);
                }
            }
        } else {
            // element i of this lane: query I*16 + g + 8*(i>>1), key J*16 + half*8 + 2*tg + (i&1)
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const int t = tq + 8 * (i >> 1), j = J * 16 + half * 8 + 2 * tg + (i & 1);
                if (j > t) continue;
                float s = 0.0f;
                for (int c = 0; c < P.dp; c++)
                    s = fmaf(to_f(sq[t * qs + c]) * to_f(sk[j * qs + c]), exp2f(sb[t * bs + c] - sb[j * bs + c]), s);
                acc[i] = s;
            }
        }
#pragma unroll
        for (int i = 0; i < 4; i += 2) {
            const int t = tq + 8 * (i >> 1), j = J * 16 + half * 8 + 2 * tg;
            float x = j <= t ? acc[i] : 0.0f, y = j + 1 <= t ? acc[i + 1] : 0.0f;
            if (!LOG) {
                x *= sb[max(t - j, 0)];
                y *= sb[max(t - j - 1, 0)];
            }
            unsigned hi, lo;
            split2(x, y, hi, lo);
            *(unsigned*)(sAh + t * as + j) = hi;
            *(unsigned*)(sAl + t * as + j) = lo;
        }
    }
    __syncthreads();

    // ---- o: warp = half of the tokens (two 16-row tiles) x a quarter of 128 value columns
    const int mt = (warp & 1) * 2, vq = warp >> 1;
    const uint4* Sin = (const uint4*)(P.ws + ((long)chunk * P.H + h) * P.dvp * P.dp);
    const int nq = P.dp >> 2;
    for (int v0 = vq * 32; v0 < P.dvp; v0 += 128) {
        float acc[2][4][4];
#pragma unroll
        for (int m = 0; m < 2; m++)
#pragma unroll
            for (int n = 0; n < 4; n++) acc[m][n][0] = acc[m][n][1] = acc[m][n][2] = acc[m][n][3] = 0.0f;
        for (int kk = 0; kk < dk; kk += 16) {
            const int c = kk + tg * 4;
            uint4 s[4];
#pragma unroll
            for (int n = 0; n < 4; n++) {
                const int v = v0 + n * 8 + g;
                s[n] = make_uint4(0, 0, 0, 0);
                if (v < P.dvp && c < P.dp) s[n] = __ldg(Sin + (long)v * nq + (c >> 2));
            }
#pragma unroll
            for (int m = 0; m < 2; m++) {
                const int t = (mt + m) * 16 + g;
                unsigned ah[4], al[4];
                if (LOG) {
                    Quad qa = load_quad(sq + t * qs + c), qb = load_quad(sq + (t + 8) * qs + c);
                    const float4 ba = *(const float4*)(sb + t * bs + c), bb = *(const float4*)(sb + (t + 8) * bs + c);
                    const float4 p = *(const float4*)(sp + (mt + m) * bs + c);
                    qa.x[0] *= exp2f(p.x + ba.x); qa.x[1] *= exp2f(p.y + ba.y); qa.x[2] *= exp2f(p.z + ba.z); qa.x[3] *= exp2f(p.w + ba.w);
                    qb.x[0] *= exp2f(p.x + bb.x); qb.x[1] *= exp2f(p.y + bb.y); qb.x[2] *= exp2f(p.z + bb.z); qb.x[3] *= exp2f(p.w + bb.w);
                    split2(qa.x[0], qa.x[1], ah[0], al[0]);
                    split2(qb.x[0], qb.x[1], ah[1], al[1]);
                    split2(qa.x[2], qa.x[3], ah[2], al[2]);
                    split2(qb.x[2], qb.x[3], ah[3], al[3]);
                } else {
                    const uint2 ua = *(const uint2*)(sq + t * qs + c), ub = *(const uint2*)(sq + (t + 8) * qs + c);
                    ah[0] = ua.x; ah[1] = ub.x; ah[2] = ua.y; ah[3] = ub.y;
                }
#pragma unroll
                for (int n = 0; n < 4; n++) {
                    mma16816(acc[m][n], ah, s[n].x, s[n].y);
                    mma16816(acc[m][n], ah, s[n].z, s[n].w);
                    if (LOG) mma16816(acc[m][n], al, s[n].x, s[n].y);
                }
            }
        }
        if (!LOG) {
#pragma unroll
            for (int m = 0; m < 2; m++) {
                const int t = (mt + m) * 16 + g;
                const float fa = sb[t + 1], fb = sb[t + 9];
#pragma unroll
                for (int n = 0; n < 4; n++) {
                    acc[m][n][0] *= fa; acc[m][n][1] *= fa;
                    acc[m][n][2] *= fb; acc[m][n][3] *= fb;
                }
            }
        }
#pragma unroll
        for (int m = 0; m < 2; m++)
            for (int J = 0; J <= mt + m; J++) {
                unsigned ah[4], al[4];
                const int off = ((mt + m) * 16 + (lane & 15)) * as + J * 16 + (lane >> 4) * 8;
                ldsm4(ah, sAh + off);
                ldsm4(al, sAl + off);
#pragma unroll
                for (int n = 0; n < 4; n += 2) {
                    const int v = v0 + n * 8;
                    if (v >= P.dvp) break;
                    unsigned r[4];
                    ldsm4t(r, sv + (J * 16 + (lane & 15)) * vs + v + (lane >> 4) * 8);
                    mma16816(acc[m][n], ah, r[0], r[1]);
                    mma16816(acc[m][n], al, r[0], r[1]);
                    mma16816(acc[m][n + 1], ah, r[2], r[3]);
                    mma16816(acc[m][n + 1], al, r[2], r[3]);
                }
            }
#pragma unroll
        for (int m = 0; m < 2; m++)
#pragma unroll
            for (int r = 0; r < 2; r++) {
                const int t = t0 + (mt + m) * 16 + g + r * 8;
                if (t >= P.T) continue;
                float* o = P.o + (long)t * P.ldo + (long)h * P.dvp;
#pragma unroll
                for (int n = 0; n < 4; n++) {
                    const int v = v0 + n * 8 + tg * 2;
                    if (v < P.dvp) *(float2*)(o + v) = make_float2(acc[m][n][2 * r], acc[m][n][2 * r + 1]);
                }
            }
    }
}

template <bool LOG>
static int launch_chunked(const ChunkP& P, cudaStream_t s) {
    const size_t sm1 = (size_t)CH * (2 * (P.dp + 8) + P.dvp + 8) * 2 + (LOG ? (size_t)CH * P.dp * 4 : CH * 4);
    const int qs = ((P.dp + 63) & ~63) + 16, bs = ((P.dp + 31) & ~31) + 16;
    const size_t sm2 = (size_t)CH * (2 * qs + P.dvp + 8 + 2 * (CH + 8)) * 2 + (LOG ? (size_t)(CH + 4) * bs * 4 : (CH + 4) * 4);
    LT_REQUIRE(sm1 <= 220 * 1024 && sm2 <= 220 * 1024, "lt_dn_recurrence_chunked: head sizes %d, %d need too much shared memory", P.dp, P.dvp);
    static PerDeviceOnce once;
    if (once.first()) {
        LT_CUDA(cudaFuncSetAttribute(k_chunk_state<LOG>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
        LT_CUDA(cudaFuncSetAttribute(k_chunk_out<LOG>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
    }
    k_chunk_state<LOG><<<dim3(P.nchunk, P.H), 256, sm1, s>>>(P);
    int rc = check_launch("lt_dn_recurrence_chunked (state)");
    if (rc != LT_OK) return rc;
    const long per = (long)P.H * P.dvp * (P.dp >> 2);
    k_chunk_scan<LOG><<<(unsigned)((per + 255) / 256), 256, 0, s>>>(P);
    rc = check_launch("lt_dn_recurrence_chunked (scan)");
    if (rc != LT_OK) return rc;
    k_chunk_out<LOG><<<dim3(P.nchunk, P.H), 256, sm2, s>>>(P);
    return check_launch("lt_dn_recurrence_chunked (out)");
}

}  // namespace dn
}  // namespace lt

using namespace lt;
using namespace lt::dn;

extern "C" long lt_dn_recurrence_chunked_ws(int T, int H, int dp, int dvp) {
    const long n = (T + CH - 1) / CH;
    return n * H * ((dp + 15) & ~15) * ((long)dvp + 1);
}

extern "C" int lt_dn_recurrence_chunked(const void* q, const void* k, const void* v, int ld, float* S, float* o, int ldo, int T, int H,
                                        int dp, int dvp, const lt_dn_decay* h_decay, float* ws, void* stream) {
    LT_REQUIRE(q && k && v && S && o && h_decay && ws, "lt_dn_recurrence_chunked: null pointer");
    LT_REQUIRE(T > 0 && H > 0 && dp > 0 && dvp > 0 && dp % 8 == 0 && dvp % 8 == 0, "lt_dn_recurrence_chunked: T=%d H=%d dp=%d dvp=%d", T, H,
               dp, dvp);
    LT_REQUIRE(dp <= 256 && dvp <= 256, "lt_dn_recurrence_chunked: head sizes %d, %d are above 256", dp, dvp);
    LT_REQUIRE(h_decay->decay || h_decay->la || h_decay->hla, "lt_dn_recurrence_chunked: decay constants or logarithms");
    LT_REQUIRE(ld % 8 == 0 && ldo % 2 == 0 && aligned16(q) && aligned16(k) && aligned16(v) && aligned16(S) && aligned16(o) && aligned16(ws),
               "lt_dn_recurrence_chunked: alignment");
    LT_REQUIRE(h_decay->decay || !h_decay->la || (h_decay->ldla % 4 == 0 && aligned16(h_decay->la)), "lt_dn_recurrence_chunked: alignment of the logarithms");
    if (!h_decay->decay && !h_decay->la) {
        SsdChunkP Q = {};
        Q.q = (const bf16*)q; Q.k = (const bf16*)k; Q.v = (const bf16*)v; Q.S = S; Q.o = o; Q.ws = ws;
        Q.hla = h_decay->hla; Q.hdt = h_decay->hdt; Q.D = h_decay->D; Q.ldh = h_decay->ldh; Q.per = h_decay->per;
        LT_REQUIRE(Q.hdt && Q.D && Q.ldh >= H && Q.per > 0 && H % Q.per == 0,
                   "lt_dn_recurrence_chunked: step sizes, D, or %d heads in groups of %d", H, Q.per);
        Q.ld = ld; Q.ldo = ldo; Q.T = T; Q.H = H; Q.dp = dp; Q.dvp = dvp; Q.nchunk = (T + CH - 1) / CH;
        return launch_ssd_chunked(Q, (cudaStream_t)stream);
    }
    ChunkP P = {};
    P.q = (const bf16*)q; P.k = (const bf16*)k; P.v = (const bf16*)v; P.S = S; P.o = o; P.ld = ld; P.ldo = ldo;
    P.T = T; P.H = H; P.dp = dp; P.dvp = dvp; P.nchunk = (T + CH - 1) / CH;
    P.ws = ws; P.dend = ws + (long)P.nchunk * H * dp * dvp;
    P.decay = h_decay->decay; P.la = h_decay->la; P.ldla = h_decay->ldla;
    if (P.decay) return launch_chunked<false>(P, (cudaStream_t)stream);
    return launch_chunked<true>(P, (cudaStream_t)stream);
}
