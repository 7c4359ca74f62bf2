/*
 * llamatov_b200_dense.h -- C ABI of libllamatov_b200_dense.so: the sm_100a kernels of models whose weights stay in
 * bfloat16 or fp32 and whose layers are mixers (linear-attention and state-space recurrences, windowed latent attention,
 * grouped-query attention) with a gated feed-forward.  Errors, the status word and the launch counter are those of libllamatov_b200_common.so
 * (llamatov_b200.h); the conventions of that header hold here too.
 *
 * Element type: `f32` = 0 means weights and activations are bfloat16 with fp32 accumulation, 1 means everything is
 * fp32 (plain fp32 fused multiply-adds; no reduced-precision matrix mode).  The residual stream, norms, decays,
 * recurrent state, attention scores and softmax weights are fp32 in both.
 * Every row length (K, leading dimensions, padded head sizes) is a multiple of 8 elements and every pointer is
 * 16-byte aligned; padding holds zeros.
 */
#ifndef LLAMATOV_B200_DENSE_H
#define LLAMATOV_B200_DENSE_H

#include "llamatov_b200.h"

#ifdef __cplusplus
extern "C" {
#endif

/* what a linear does with v = (W x)[n] (+ bias[n]) */
#define LT_DN_STORE 0 /* y = act(v) * scale, per output segment */
#define LT_DN_RESID 1 /* y (fp32) += ls[n] * v; ls may be NULL (1) */
#define LT_DN_GLU 2   /* rows n and n + M of W are gate and up: y = glu(v_gate, v_up), M outputs */
#define LT_DN_STORE_GLU 3 /* lt_dn_gemv only: rows below glu_from as LT_DN_STORE, then M - glu_from gate and as many up
                             rows as LT_DN_GLU, whose outputs go to y2 */

#define LT_DN_GLU_GELU 0    /* gelu_tanh(g) * u */
#define LT_DN_GLU_CLAMPED 1 /* g = min(g, limit), u = clamp(u, -limit, limit): g * sigmoid(alpha g) * (u + 1) */

#define LT_DN_ACT_NONE 0
#define LT_DN_ACT_SILU 1
#define LT_DN_ACT_SIGMOID 2
#define LT_DN_ACT_LOGSIGMOID 3

#define LT_DN_MAX_SEG 6

typedef struct {
    int kind;
    int out_f32;                  /* LT_DN_STORE / LT_DN_GLU: store fp32 instead of the element type */
    int nseg;                     /* 0 = no activation, scale 1 */
    int seg_end[LT_DN_MAX_SEG];   /* outputs [seg_end[i-1], seg_end[i]) get act and scale i */
    int seg_act[LT_DN_MAX_SEG];
    float seg_scale[LT_DN_MAX_SEG];
    const float* bias;            /* [M] or NULL */
    const float* ls;              /* [M] or NULL */
    int glu_act;
    float glu_alpha, glu_limit;
    int tail_from, ldtail;        /* LT_DN_STORE with tail: outputs n >= tail_from go in fp32 to tail[t][n - tail_from] */
    float* tail;                  /* or NULL */
    int glu_from;
    void* y2;
} lt_dn_epilogue;

#define LT_DN_IN_TYPED 0 /* x: K elements of the element type */
#define LT_DN_IN_CAST 1  /* fp32 x [n1], then fp32 x2 [K - n1] (x2 may be NULL when n1 == K) */
#define LT_DN_IN_NORM 2  /* fp32 x [n1] in groups: x / sqrt(sum / count + eps) * w (* gate), then K - n1 elements of the
                            element type from x2 (n1 = 0 means K) */

typedef struct {
    int kind;
    int n1;
    int group, count;   /* LT_DN_IN_NORM: elements per group (padded) and how many of them count in the mean */
    float eps;
    const void* x;
    const void* x2;
    const float* w;     /* [w_period], index = position modulo w_period */
    int w_period;
    const void* gate;   /* n1 elements of the element type, or NULL */
    int gate_first;     /* the gate multiplies x ahead of the norm instead of the normed value */
    int seg, segp;      /* seg > 0: the vector is segments of segp elements of which seg are real, and a group is `count`
                           consecutive real elements wherever the segments end (w has n1 entries then) */
} lt_dn_prologue;

/* x[t][0..ld) = table[tok[t]][0..E) * scale in fp32, zeros from E to ld; x0 (or NULL) gets the same rows.  With norm_w
 * [E] (or NULL) the row is then RMS-normed: v / sqrt(mean(v^2) + eps) * norm_w. */
int lt_dn_embed(const void* table, int f32, int tab_ld, const int* tok, float scale, const float* norm_w, float eps, float* x,
                float* x0, int E, int ld, int V, int T, void* stream);

/* rows of fp32 x in groups of `group` elements: y = x / sqrt(sum / count + eps) * w (* gate), stored in the element
 * type.  rows (or NULL): row t reads x row rows[t].  gate_first, seg, segp as in lt_dn_prologue. */
int lt_dn_norm_rows(const float* x, int ldx, const int* rows, const float* w, int w_period, const void* gate, int ldg,
                    void* y, int ldy, int f32, int T, int N, int group, int count, float eps, int gate_first, int seg, int segp,
                    void* stream);

/* y[t] = [x[t], x2[t]] cast to the element type, n1 and n2 columns */
int lt_dn_concat_rows(const float* x, int ldx, int n1, const float* x2, int ldx2, int n2, void* y, int ldy, int f32, int T,
                      void* stream);

/* Y[t][n] = epilogue((W x_t)[n]) for T rows.  bf16: tcgen05 tiles; fp32: CUDA cores.  `variant` 0 = choose the tile,
 * else the tile's token columns (32, 64, 128 or 256; 256 not for LT_DN_GLU). */
int lt_dn_linear(const void* W, int ldw, const void* X, int ldx, void* Y, int ldy, int f32, int M, int K, int T,
                 const lt_dn_epilogue* h_epi, int variant, void* stream);

/* The same for one row, whose input is made by a prologue in every CTA (norm, gate, cast). */
int lt_dn_gemv(const void* W, int ldw, void* Y, int f32, int M, int K, const lt_dn_prologue* h_pro,
               const lt_dn_epilogue* h_epi, void* stream);

/* Linear-attention recurrence of H heads, in token order:
 *   S <- diag(a_t) S + k_t v_t^T,  o_t = S^T q_t        (S fp32, stored [H][dvp][dp], updated in place)
 * q, k, v: element type, row stride ld, head h at columns h*dp (q, k) and h*dvp (v); o: fp32, row stride ldo.
 * The decay a_t comes from exactly one of: decay [H] (one constant per head); la [T][ldla] fp32, the logarithms per
 * key channel, head h at h*dp; or, for T = 1, a1 [rank] (element type) with a2 [H*dp][lda2], bias [H*dp]:
 * log a = logsigmoid(a2 a1 + bias) * inv_tau; or the state-space form, hla [T][ldh] fp32 with hdt [T][ldh] and D [H]:
 *   S <- exp(hla_t) S + hdt_t k_t v_t^T,  o_t = S^T q_t + D v_t,   q and k shared by `per` consecutive heads. */
typedef struct {
    const float* decay;
    const float* la;
    int ldla;
    const void* a1;
    const void* a2;
    int lda2, rank;
    const float* bias;
    float inv_tau;
    const float* hla;
    const float* hdt;
    const float* D;
    int ldh, per;
} lt_dn_decay;

int lt_dn_recurrence(const void* q, const void* k, const void* v, int ld, float* S, float* o, int ldo, int f32, int T,
                     int H, int dp, int dvp, const lt_dn_decay* h_decay, void* stream);

/* The same over a prompt portion in chunks on the tensor cores (bf16 only; la, decay or hla).  ws: fp32 workspace of
 * lt_dn_recurrence_chunked_ws(T, H, dp, dvp) elements. */
long lt_dn_recurrence_chunked_ws(int T, int H, int dp, int dvp);
int lt_dn_recurrence_chunked(const void* q, const void* k, const void* v, int ld, float* S, float* o, int ldo, int T,
                             int H, int dp, int dvp, const lt_dn_decay* h_decay, float* ws, void* stream);

/* Windowed latent attention.  Per position the cache keeps one row [c (rp), rotated key part (rtp)], at slot
 * position % cap of a ring. */
typedef struct {
    int H, dp, rtp, dvp;  /* padded per-head sizes: unrotated, rotated, value */
    int rot;              /* rotated dimensions: i is paired with i + rot/2 */
    int rp, rank;         /* padded and true latent size */
    int window, cap;
    float scale, eps;
    const float* freq;    /* [rot/2] */
    const float* cnorm;   /* [rp] */
} lt_dn_latent;

/* T rows at positions pos0 ..: y rows are [q heads: H * (dp + rtp) | c: rp | kr: rtp], row stride ld.  Rotates q in
 * place, norms c, rotates kr, stores the row in the ring and in rows np .. of `keys` [np + T][rp + rtp]; rows 0 .. np-1
 * of keys are copied from the ring (positions pos0 - np ..). */
int lt_dn_latent_rows(void* y, int ld, void* ring, void* keys, int np, int pos0, int f32, int T, const lt_dn_latent* h_l,
                      void* stream);

/* out[t][h*dvp ..] = softmax over the window of ((q . k) * scale) v for T queries at positions np .. np+T-1 relative
 * to the first of the nk = np + T keys; kn and v are the expanded keys and values (row strides ldkn, ldv), kr the
 * shared rotated part (row stride ldkr). */
int lt_dn_window_attn(const void* q, int ldq, const void* kn, int ldkn, const void* kr, int ldkr, const void* v, int ldv,
                      void* out, int ldo, int f32, int T, int np, const lt_dn_latent* h_l, void* stream);

/* One token at position *len (then *len += 1), keys and values left in latent form: q_abs = W_uk^T q, the window is
 * scanned over cache rows by `splits` CTAs per head group, the value projection follows the sum over positions.
 * y: one row as in lt_dn_latent_rows.  ukT [H][rp][dp], uv [H*dvp][rp].  out: H*dvp elements.
 * ws: lt_dn_latent_step_ws(H, rp, rtp, splits) fp32 elements. */
long lt_dn_latent_step_ws(int H, int rp, int rtp, int splits);
int lt_dn_latent_step(const void* y, void* ring, int* len, const void* ukT, const void* uv, void* out, int f32,
                      const lt_dn_latent* h_l, int splits, float* ws, void* stream);

/* State-space mixer: a recurrence with step sizes per token and head, behind a short convolution.
 * From `xbc` on a row holds C = H*dvp + 2*G*dp channels that pass a causal convolution of `taps` taps per channel and silu: x
 * (H*dvp), then keys and queries of G groups (G*dp each).  The convolution's last inputs are kept in a ring [taps][C] of the
 * element type, position p in row p % taps. */
typedef struct {
    int H, G, dp, dvp, taps;
    const float* conv;     /* [taps][C]; the last tap is the current token's */
    const float* conv_b;   /* [C] */
    const float* dt_bias;  /* [H] */
    const float* A;        /* [H]: log decay per unit of step size (negative) */
    const float* D;        /* [H] */
} lt_dn_ssd;

/* T rows at positions pos0 ..: out [T][ldo] = silu(conv + bias), hdt = softplus(dt + dt_bias), hla = A * hdt ([T][H] fp32; dt
 * [T][lddt] fp32); then the ring takes the portion's last inputs (two launches). */
int lt_dn_ssd_rows(const void* xbc, int ld, const float* dt, int lddt, void* ring, void* out, int ldo, float* hla, float* hdt,
                   int f32, int T, int pos0, const lt_dn_ssd* h_s, void* stream);

/* One token at position *len (then *len += 1): convolution, step size and recurrence in one launch.  S [H][dvp][dp] fp32, o
 * [H*dvp] fp32.  ticket: one int, zero between launches. */
int lt_dn_ssd_step(const void* xbc, const float* dt, void* ring, float* S, float* o, int f32, int* len, int* ticket,
                   const lt_dn_ssd* h_s, void* stream);

/* Grouped-query attention over all earlier positions.  The cache keeps k [cap][G*dp] and v [cap][G*dvp] of the element
 * type, position p in row p. */
typedef struct {
    int H, G, dp, dvp;     /* query heads, key/value heads, padded head sizes */
    int rot;               /* rotated dimensions of a head: i is paired with i + rot/2 */
    int qcount, kcount;    /* real elements of all queries / all keys (the norms' means) */
    int cap;               /* rows of the cache */
    float scale, softcap, eps;   /* softcap 0: none; else score <- softcap * tanh(score / softcap) */
    float vmix;            /* v <- (1 - vmix) v + vmix * vfirst where vfirst is given */
    const float* freq;     /* [rot/2][2]: a frequency as the sum of two floats */
    const float* qnorm;    /* [H*dp] */
    const float* knorm;    /* [G*dp] */
} lt_dn_gqa;

/* T rows at positions pos0 ..: y rows are [q: H*dp | k: G*dp | v: G*dvp ...], row stride ld.  Norms q and k over the whole
 * projection, rotates them, mixes v; q is replaced, k and v go to the cache.  vfirst [T][G*dvp] or NULL: with vmix_store the
 * row's own v is written there instead of being mixed. */
int lt_dn_gqa_rows(void* y, int ld, void* kc, void* vc, void* vfirst, int vmix_store, int f32, int T, int pos0,
                   const lt_dn_gqa* h_a, void* stream);

/* out[t][h*dvp ..] = gate[t][h] * softmax over positions <= np + t of score(q, k) v for T queries at positions np .. (gate:
 * fp32 or NULL). */
int lt_dn_gqa_attn(const void* q, int ldq, const void* kc, const void* vc, const float* gate, int ldg, void* out, int ldo, int f32,
                   int T, int np, const lt_dn_gqa* h_a, void* stream);

/* One token at position *len (then *len += 1), in one launch: norms, rotation, value mixing, append, scores over `splits`
 * ranges of positions per key head, combination, gate.  y: one row as in lt_dn_gqa_rows (not changed); gate [H] fp32 or NULL.
 * ws: lt_dn_gqa_step_ws(H, dvp, splits) fp32 elements; tickets: lt_dn_gqa_step_tickets(H, G) ints, zero between launches. */
long lt_dn_gqa_step_ws(int H, int dvp, int splits);
int lt_dn_gqa_step_tickets(int H, int G);
int lt_dn_gqa_step(const void* y, void* kc, void* vc, void* vfirst, int vmix_store, const float* gate, void* out, int f32, int* len,
                   const lt_dn_gqa* h_a, int splits, float* ws, int* tickets, void* stream);

#ifdef __cplusplus
}
#endif
#endif
