// Linear over a block of token rows, Y[t][n] = epilogue(sum_k W[n][k] X[t][k]).
//
// bf16 (k_gemm_tc): tcgen05.mma kind::f16, fp32 accumulators in tensor memory.  A tile is MA x 128 weight rows (the
// MMA's M: tensor-memory lanes) by NT tokens (its N: columns); with MA = 2 the second 128 rows are the "up" rows that
// belong to the first 128 "gate" rows, so that act(gate) * up is formed where both accumulators are.  An epilogue
// thread owns one weight row: bias, activation and layer scale are per-thread constants, and the 32 lanes of a
// warp store 32 consecutive outputs of a token.
//   warp 8 : producer, TMA tiles of 64 k (128-byte rows, hardware swizzle) into a ring of shared-memory stages
//   warp 9 : one thread issues the MMAs; two accumulator sets, so the next tile's MMAs run under this tile's epilogue
//   warps 0-7 : epilogue
// fp32 (k_gemm_f32): 64 x 64 tiles on the CUDA cores, every product and sum an fp32 fused multiply-add.
#include "lt_dn_common.cuh"
#include "lt_tc.cuh"

namespace lt {
namespace dn {

using namespace tc;

struct GemmP {
    void* Y;
    int* status;
    int M, K, T, ldy;
    int row_tiles, t_tiles;
    int up_row;          // first "up" row (MA = 2)
    lt_dn_epilogue epi;
};

constexpr int BK = 64;   // k elements of a stage (128 bytes)

template <int NT, int MA>
struct GemmCfg {
    static constexpr int W_STAGE = MA * 128 * 128;
    static constexpr int X_STAGE = NT * 128;
    static constexpr int STAGE = W_STAGE + X_STAGE;
    static constexpr int NSTAGE = (200 * 1024) / STAGE > 8 ? 8 : (200 * 1024) / STAGE;
    static constexpr int ACC_COLS = MA * NT;
    static constexpr int TMEM = 2 * ACC_COLS < 32 ? 32 : 2 * ACC_COLS;
    static constexpr int EW = 8;
    static constexpr int THREADS = (EW + 2) * 32;
    static constexpr int SMEM = 1024 + NSTAGE * STAGE + 1024;
    static_assert(TMEM <= 512 && (TMEM & (TMEM - 1)) == 0, "tensor memory columns");
    static_assert(X_STAGE % 1024 == 0, "stages keep 1024-byte alignment");
};

struct GemmBars {
    unsigned long long full[8], empty[8], tfull[2], tempty[2];
    unsigned tmem_base;
    int abort_flag;
};

// D[tmem] (+)= A[smem] * B[smem], bf16 x bf16 -> fp32
__device__ __forceinline__ void mma_bf16(unsigned d, unsigned long long a, unsigned long long b, unsigned idesc, bool acc) {
    asm volatile(
        "{\n\t.reg .pred p;\n\t"
        "setp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}" ::"r"(d),
        "l"(a), "l"(b), "r"(idesc), "r"((int)acc)
        : "memory");
}

template <int NT, int MA>
__global__ void __launch_bounds__(GemmCfg<NT, MA>::THREADS, 1)
k_gemm_tc(const __grid_constant__ CUtensorMap tmW, const __grid_constant__ CUtensorMap tmX, const __grid_constant__ GemmP P) {
    using C = GemmCfg<NT, MA>;
    constexpr int NS = C::NSTAGE;
    extern __shared__ __align__(1024) unsigned char smem_raw[];
    unsigned char* base = (unsigned char*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    GemmBars* B = (GemmBars*)(base + NS * C::STAGE);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int tiles = P.row_tiles * P.t_tiles;
    const int nk = (P.K + BK - 1) / BK;
    volatile int* abort_flag = &B->abort_flag;

    if (tid == 0) {
        for (int s = 0; s < NS; s++) {
            mbar_init(&B->full[s], 1);
            mbar_init(&B->empty[s], 1);
        }
        for (int s = 0; s < 2; s++) {
            mbar_init(&B->tfull[s], 1);
            mbar_init(&B->tempty[s], C::EW);
        }
        B->abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == C::EW + 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&B->tmem_base)),
                     "r"((unsigned)C::TMEM)
                     : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const unsigned tmem = B->tmem_base;

    if (warp == C::EW) {
        if (lane == 0) {
            unsigned it = 0;
            for (int tile = blockIdx.x; tile < tiles; tile += gridDim.x) {
                const int rt = tile % P.row_tiles, tt = tile / P.row_tiles;
                for (int kb = 0; kb < nk; kb++, it++) {
                    const int s = it % NS;
                    unsigned char* st = base + s * C::STAGE;
                    mbar_wait<32>(&B->empty[s], ((it / NS) & 1) ^ 1, abort_flag, P.status);
                    mbar_expect_tx(&B->full[s], C::STAGE);
                    tma_load_2d(st, &tmW, kb * BK, rt * 128, &B->full[s]);
                    if (MA == 2) tma_load_2d(st + 128 * 128, &tmW, kb * BK, P.up_row + rt * 128, &B->full[s]);
                    tma_load_2d(st + C::W_STAGE, &tmX, kb * BK, tt * NT, &B->full[s]);
                }
            }
        }
    } else if (warp == C::EW + 1) {
        if (lane == 0) {
            // D fp32, A and B bf16, both K-major, N = NT, M = 128
            constexpr unsigned idesc =
                (1u << 4) | (1u << 7) | (1u << 10) | ((unsigned)(NT >> 3) << 17) | ((unsigned)(128 >> 4) << 24);
            const unsigned long long w0 = smem_desc<4>(smem_u32(base));
            const unsigned long long x0 = smem_desc<4>(smem_u32(base) + C::W_STAGE);
            unsigned it = 0, n = 0;
            for (int tile = blockIdx.x; tile < tiles; tile += gridDim.x, n++) {
                const unsigned slot = n & 1;
                mbar_wait<32>(&B->tempty[slot], ((n >> 1) & 1) ^ 1, abort_flag, P.status);
                tc_fence_after();
                const unsigned d = tmem + slot * C::ACC_COLS;
                for (int kb = 0; kb < nk; kb++, it++) {
                    const unsigned s = it % NS;
                    mbar_wait<0>(&B->full[s], (it / NS) & 1, abort_flag, P.status);
                    tc_fence_after();
                    const unsigned long long wd = w0 + (unsigned long long)(s * (C::STAGE >> 4));
                    const unsigned long long xd = x0 + (unsigned long long)(s * (C::STAGE >> 4));
#pragma unroll
                    for (int j = 0; j < BK / 16; j++) {
#pragma unroll
                        for (int a = 0; a < MA; a++)
                            mma_bf16(d + a * NT, wd + a * (128 * 128 >> 4) + 2 * j, xd + 2 * j, idesc, kb > 0 || j > 0);
                    }
                    mma_commit(&B->empty[s]);
                }
                mma_commit(&B->tfull[slot]);
            }
        }
    } else {
        const int q = warp & 3, cg = warp >> 2;
        constexpr int CW = NT / 2;                // columns of this warp
        unsigned n = 0;
        for (int tile = blockIdx.x; tile < tiles; tile += gridDim.x, n++) {
            const int rt = tile % P.row_tiles, tt = tile / P.row_tiles;
            const int row = rt * 128 + q * 32 + lane;
            const bool row_ok = row < P.M;
            const int t0 = tt * NT + cg * CW;
            const unsigned slot = n & 1;
            const RowEpi re = row_epi(P.epi, row_ok ? row : 0);
            mbar_wait<32>(&B->tfull[slot], (n >> 1) & 1, abort_flag, P.status);
            tc_fence_after();
            const unsigned ta = tmem + ((unsigned)(q * 32) << 16) + slot * C::ACC_COLS + cg * CW;
#pragma unroll 1
            for (int c0 = 0; c0 < CW; c0 += 16) {
                if (t0 + c0 >= P.T) break;        // the same for the whole warp
                int v[MA][16];
#pragma unroll
                for (int a = 0; a < MA; a++) tmem_ld<16>(ta + a * NT + c0, v[a]);
                asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
                for (int a = 0; a < MA; a++)
#pragma unroll
                    for (int c = 0; c < 16; c += 4) reg_fence4(&v[a][c]);
                if (row_ok) {
                    if (MA == 2) {
                        float f[16];
                        if (P.epi.out_f32) {
#pragma unroll
                            for (int c = 0; c < 16; c++)
                                f[c] = glu_f(P.epi, __int_as_float(v[0][c]), __int_as_float(v[MA - 1][c]));
                            float* y = (float*)P.Y + (long)(t0 + c0) * P.ldy + row;
#pragma unroll
                            for (int c = 0; c < 16; c++)
                                if (t0 + c0 + c < P.T) y[(long)c * P.ldy] = f[c];
                        } else {
                            glu_bf16(P.epi, v[0], v[MA - 1], f);
                            bf16* y = (bf16*)P.Y + (long)(t0 + c0) * P.ldy + row;
#pragma unroll
                            for (int c = 0; c < 16; c++)
                                if (t0 + c0 + c < P.T) y[(long)c * P.ldy] = from_f<bf16>(f[c]);
                        }
                    } else if (P.epi.kind == LT_DN_RESID) {
                        float* y = (float*)P.Y + (long)(t0 + c0) * P.ldy + row;
                        float old[16];
#pragma unroll
                        for (int c = 0; c < 16; c++)
                            if (t0 + c0 + c < P.T) old[c] = y[(long)c * P.ldy];
#pragma unroll
                        for (int c = 0; c < 16; c++)
                            if (t0 + c0 + c < P.T)
                                y[(long)c * P.ldy] = fmaf(re.ls, __int_as_float(v[0][c]) + re.bias, old[c]);
                    } else {
                        float f[16];
#pragma unroll
                        for (int c = 0; c < 16; c++) f[c] = __int_as_float(v[0][c]);
                        if (P.epi.tail != nullptr && row >= P.epi.tail_from) {
                            epi_values<false>(re, f);
                            float* y = P.epi.tail + (long)(t0 + c0) * P.epi.ldtail + row - P.epi.tail_from;
#pragma unroll
                            for (int c = 0; c < 16; c++)
                                if (t0 + c0 + c < P.T) y[(long)c * P.epi.ldtail] = f[c];
                        } else if (P.epi.out_f32) {
                            epi_values<false>(re, f);
                            float* y = (float*)P.Y + (long)(t0 + c0) * P.ldy + row;
#pragma unroll
                            for (int c = 0; c < 16; c++)
                                if (t0 + c0 + c < P.T) y[(long)c * P.ldy] = f[c];
                        } else {
                            epi_values<true>(re, f);
                            bf16* y = (bf16*)P.Y + (long)(t0 + c0) * P.ldy + row;
#pragma unroll
                            for (int c = 0; c < 16; c++)
                                if (t0 + c0 + c < P.T) y[(long)c * P.ldy] = from_f<bf16>(f[c]);
                        }
                    }
                }
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&B->tempty[slot]);
        }
    }

    tc_fence_before();
    __syncthreads();
    if (*abort_flag && tid == 0) {     // a wait ran out: let copies in flight land before the CTA leaves
        const long long t0 = clock64();
        while (clock64() - t0 < 2000000LL) {
        }
    }
    __syncthreads();
    if (warp == C::EW + 1) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"((unsigned)C::TMEM) : "memory");
    }
}

// [rows][K] bf16 with row stride ld, box 64 k x box_rows
static int make_map_bf16(CUtensorMap* m, const void* ptr, long rows, int K, int ld, int box_rows) {
    encode_fn_t fn = encode_fn();
    if (fn == nullptr) {
        set_error("lt_dn_linear: cuTensorMapEncodeTiled is not available from this driver");
        return LT_ERR_CUDA;
    }
    cuuint64_t dims[2] = {(cuuint64_t)K, (cuuint64_t)rows};
    cuuint64_t strides[1] = {(cuuint64_t)ld * 2};
    cuuint32_t box[2] = {(cuuint32_t)BK, (cuuint32_t)box_rows};
    cuuint32_t estr[2] = {1, 1};
    CUresult r = fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(ptr), dims, strides, box, estr,
                    CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B,
                    CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) {
        set_error("lt_dn_linear: cuTensorMapEncodeTiled failed (%d) for rows=%ld K=%d ld=%d", (int)r, rows, K, ld);
        return LT_ERR_CUDA;
    }
    return LT_OK;
}

template <int NT, int MA>
static int launch_tc(const void* W, int ldw, const void* X, int ldx, GemmP P, cudaStream_t s) {
    using C = GemmCfg<NT, MA>;
    CUtensorMap tmW, tmX;
    int rc = make_map_bf16(&tmW, W, (long)P.M * MA, P.K, ldw, 128);
    if (rc != LT_OK) return rc;
    rc = make_map_bf16(&tmX, X, P.T, P.K, ldx, NT);
    if (rc != LT_OK) return rc;
    static PerDeviceOnce once;
    if (once.first())
        LT_CUDA(cudaFuncSetAttribute(k_gemm_tc<NT, MA>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM));
    P.row_tiles = (P.M + 127) / 128;
    P.t_tiles = (P.T + NT - 1) / NT;
    P.up_row = P.M;
    P.status = device_status_ptr();
    LT_REQUIRE(P.status != nullptr, "lt_dn_linear: status word unavailable");
    const long tiles = (long)P.row_tiles * P.t_tiles;
    const int sms = sm_count();
    k_gemm_tc<NT, MA><<<(int)(tiles < sms ? tiles : sms), C::THREADS, C::SMEM, s>>>(tmW, tmX, P);
    return check_launch("lt_dn_linear");
}

// ---------------------------------------------------------------------------- fp32

// thread (tx, ty): outputs n = 4 groups of 16 apart, so that a warp's stores are contiguous
template <bool GLU>
__global__ void __launch_bounds__(256) k_gemm_f32(const float* __restrict__ W, int ldw, const float* __restrict__ X, int ldx,
                                                  const __grid_constant__ GemmP P) {
    __shared__ float sw[GLU ? 2 : 1][16][65], sx[16][65];
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    const int n0 = blockIdx.x * 64, t0 = blockIdx.y * 64;
    float acc[GLU ? 2 : 1][4][4];
#pragma unroll
    for (int g = 0; g < (GLU ? 2 : 1); g++)
#pragma unroll
        for (int i = 0; i < 4; i++)
#pragma unroll
            for (int j = 0; j < 4; j++) acc[g][i][j] = 0.0f;
    const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;     // row and first k this thread loads
    for (int k0 = 0; k0 < P.K; k0 += 16) {
        const bool k_ok = k0 + lk < P.K;                             // K is a multiple of 4
#pragma unroll
        for (int g = 0; g < (GLU ? 2 : 1); g++) {
            float4 w = make_float4(0, 0, 0, 0);
            if (k_ok && n0 + lr < P.M) w = *(const float4*)(W + (long)(g * P.up_row + n0 + lr) * ldw + k0 + lk);
            sw[g][lk][lr] = w.x; sw[g][lk + 1][lr] = w.y; sw[g][lk + 2][lr] = w.z; sw[g][lk + 3][lr] = w.w;
        }
        float4 x = make_float4(0, 0, 0, 0);
        if (k_ok && t0 + lr < P.T) x = *(const float4*)(X + (long)(t0 + lr) * ldx + k0 + lk);
        sx[lk][lr] = x.x; sx[lk + 1][lr] = x.y; sx[lk + 2][lr] = x.z; sx[lk + 3][lr] = x.w;
        __syncthreads();
#pragma unroll
        for (int k = 0; k < 16; k++) {
            float b[4];
#pragma unroll
            for (int j = 0; j < 4; j++) b[j] = sx[k][ty + 16 * j];
#pragma unroll
            for (int g = 0; g < (GLU ? 2 : 1); g++)
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    const float a = sw[g][k][tx + 16 * i];
#pragma unroll
                    for (int j = 0; j < 4; j++) acc[g][i][j] = fmaf(a, b[j], acc[g][i][j]);
                }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const int n = n0 + tx + 16 * i;
        if (n >= P.M) continue;
        const RowEpi re = row_epi(P.epi, n);
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int t = t0 + ty + 16 * j;
            if (t >= P.T) continue;
            if (GLU) glu_store<float>(P.epi, P.Y, (long)t * P.ldy + n, acc[0][i][j], acc[GLU ? 1 : 0][i][j]);
            else epi_store<float>(P.epi, re, P.Y, t, P.ldy, n, acc[0][i][j]);
        }
    }
}

// tile width: fewest (waves x time of a tile); a tile costs its columns plus what does not shrink with them
static int choose_nt(int M, int T, bool glu) {
    const int sms = sm_count();
    const int cand[4] = {256, 128, 64, 32};
    int best = 32;
    double cost = 1e30;
    for (int i = glu ? 1 : 0; i < 4; i++) {
        const long tiles = (long)((M + 127) / 128) * ((T + cand[i] - 1) / cand[i]);
        const double c = (double)((tiles + sms - 1) / sms) * ((glu ? 2 : 1) * cand[i] + 48);
        if (c < cost) {
            cost = c;
            best = cand[i];
        }
    }
    return best;
}

}  // namespace dn
}  // namespace lt

using namespace lt;
using namespace lt::dn;

extern "C" int lt_dn_linear(const void* W, int ldw, const void* X, int ldx, void* Y, int ldy, int f32, int M, int K, int T,
                            const lt_dn_epilogue* h_epi, int variant, void* stream) {
    LT_REQUIRE(W && X && Y, "lt_dn_linear: null pointer");
    const char* bad = epi_error(h_epi);
    LT_REQUIRE(bad == nullptr, "lt_dn_linear: %s", bad);
    LT_REQUIRE(M > 0 && T > 0 && K > 0 && K % 8 == 0, "lt_dn_linear: M=%d T=%d K=%d (K a multiple of 8)", M, T, K);
    LT_REQUIRE(ldw >= K && ldw % 8 == 0 && ldx >= K && ldx % 8 == 0, "lt_dn_linear: ldw=%d ldx=%d must be multiples of 8, >= K=%d",
               ldw, ldx, K);
    const int my = h_epi->kind == LT_DN_STORE && h_epi->tail != nullptr && h_epi->tail_from < M ? h_epi->tail_from : M;
    LT_REQUIRE(ldy >= my, "lt_dn_linear: ldy=%d < M=%d", ldy, my);
    LT_REQUIRE(h_epi->kind != LT_DN_STORE_GLU, "lt_dn_linear: the combined epilogue is lt_dn_gemv's");
    LT_REQUIRE(aligned16(W) && aligned16(X), "lt_dn_linear: W and X must be 16-byte aligned");
    LT_REQUIRE(variant == 0 || variant == 32 || variant == 64 || variant == 128 || variant == 256,
               "lt_dn_linear: unknown variant %d", variant);
    cudaStream_t s = (cudaStream_t)stream;
    GemmP P = {};
    P.Y = Y; P.M = M; P.K = K; P.T = T; P.ldy = ldy; P.epi = *h_epi; P.up_row = M;
    const bool glu = h_epi->kind == LT_DN_GLU;
    if (f32) {
        dim3 grid((M + 63) / 64, (T + 63) / 64);
        LT_REQUIRE(grid.y <= 65535, "lt_dn_linear: T=%d too large", T);
        if (glu) k_gemm_f32<true><<<grid, 256, 0, s>>>((const float*)W, ldw, (const float*)X, ldx, P);
        else k_gemm_f32<false><<<grid, 256, 0, s>>>((const float*)W, ldw, (const float*)X, ldx, P);
        return check_launch("lt_dn_linear");
    }
    const int nt = variant ? variant : choose_nt(M, T, glu);
    if (glu) {
        LT_REQUIRE(nt <= 128, "lt_dn_linear: tiles of 256 tokens do not fit a gated pair");
        if (nt == 128) return launch_tc<128, 2>(W, ldw, X, ldx, P, s);
        if (nt == 64) return launch_tc<64, 2>(W, ldw, X, ldx, P, s);
        return launch_tc<32, 2>(W, ldw, X, ldx, P, s);
    }
    if (nt == 256) return launch_tc<256, 1>(W, ldw, X, ldx, P, s);
    if (nt == 128) return launch_tc<128, 1>(W, ldw, X, ldx, P, s);
    if (nt == 64) return launch_tc<64, 1>(W, ldw, X, ldx, P, s);
    return launch_tc<32, 1>(W, ldw, X, ldx, P, s);
}
