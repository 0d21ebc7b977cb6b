/* scmx_mixers.h — C ABI of libscmx_mixers.so: sequence mixers and bfloat16 / float32 matrix products of the hybrid decoder
 * models (selective scan, retention, differential attention, gated delta rules, latent attention) on NVIDIA B200 (sm_100a).
 *
 * Conventions are those of scmx.h: device pointers only, nothing is allocated, work is enqueued on `stream`, 0 on success,
 * shapes are validated on the host.  Additional ones:
 *   - `dt` names the storage type of the activations, weights or cache concerned: 0 = bfloat16, 1 = float32.  Norms, scores,
 *     recurrences and the residual stream are float32 in both cases.
 *   - "ld" arguments are row pitches in elements.  Small per-channel vectors (norm weights, biases, decays) are float32.
 *   - A position on the device (`pos_dev`, int32, may be NULL) replaces the host-side position, so that a captured decode step
 *     can be replayed while the sequence grows.
 * The functions have no counterpart in the reference project.
 */
#ifndef SCMX_MIXERS_H_
#define SCMX_MIXERS_H_

#include "scmx.h"

#ifdef __cplusplus
extern "C" {
#endif

/* x[t] = table[tokens[t]] (float32) and the same row in storage type as h (NULL: not wanted). */
int scmx_embed(const int64_t* tokens, const void* table, int dt, int64_t V, int64_t T, int W, float* x, void* h, void* stream);

/* x[t] = scale table[tokens[t]] + pairs[row] (pairs NULL: no second table), row = (token before * mul_prev + token * mul_cur) mod
 * buckets, and row `buckets` where there is no token before.  prev: the token before this portion (negative: none), advanced. */
int scmx_embed_pair(const int64_t* tokens, const void* table, const void* pairs, int dt, int64_t V, int64_t T, int W, float scale,
                    int64_t buckets, int64_t mul_prev, int64_t mul_cur, int64_t* prev, float* x, void* stream);

/* x_out = x + mult * y and h_out = x_out / rms(x_out) * w in storage type dt (y NULL: only the norm of x).  x_out may be x. */
int scmx_add_norm(const float* y, int64_t ldy, const float* x, const float* w, float mult, float eps, int64_t T, int W, float* x_out,
                  void* h_out, int dt, void* stream);

/* r = x + w * y / rms(y).  n = 0: x_out = r.  n > 0: x_out = sum_{j < n-1} dwa[j] xs[j] + dwa[n-1] r, and with keep xs[n-1] = r
 * (xs: [n][T, W] results xs_stride elements apart).  h_out: x_out in storage type dt, or NULL.  x_out may be x. */
int scmx_res_norm(const float* y, int64_t ldy, const float* x, const float* w, float eps, int64_t T, int W, float* xs, int64_t xs_stride,
                  const float* dwa, int n, int keep, float* x_out, void* h_out, int dt, void* stream);

/* out[m] = w * x[rows[m]] / rms (rows NULL: m itself). */
int scmx_norm_rows(const float* x, const int64_t* rows, const float* w, float eps, int64_t M, int W, void* out, int dt, void* stream);

/* Causal depthwise convolution + SiLU: w [C, taps] (last column: the current token), b [C] or NULL; tail [C, taps-1] holds the inputs
 * before this portion, oldest first, and is advanced. */
int scmx_conv_silu(const void* x, int64_t ldx, int dt, int64_t T, int C, int taps, const float* w, const float* b, float* tail, void* out,
                   int64_t ldo, void* stream);

/* out[t, h] = o[t, h] / rms(o[t, h]) * w * gate(g[t, h]), dv values per head, w [dv] or NULL; gate: 0 = SiLU, 1 = sigmoid. */
int scmx_head_norm_gate(const float* o, const void* g, int64_t ldg, int dt, const float* w, int gate, int64_t T, int H, int dv, float eps,
                        void* out, void* stream);

/* out [rows, n] = gelu(gate) up (tanh form) of rows whose columns alternate 16 gate and 16 up values; n a multiple of 16. */
int scmx_gated_gelu(const float* x, int64_t ldx, int64_t rows, int n, float* out, void* stream);

/* In place on n float32 values: softplus(p) z^2 + z/2 above zero, (1/2 + softplus(q)) (e^z - 1 - z) + z/2 below. */
int scmx_xielu(float* x, int64_t n, float a_pos, float a_neg, void* stream);

/* Selective scan over n tokens: step = softplus(dtp + dt_bias), S <- 2^(step A2) S + step x B, y = (S C + D x) silu(z).
 * A2 = -exp(A_log) log2(e) [C, N]; bc holds B at column 0 and C at column N; state [C, N] is carried. */
int scmx_selective_scan(const void* x, int64_t ldx, const float* dtp, int64_t ldt, const void* bc, int64_t ldbc, const void* z, int64_t ldz,
                        int dt, int64_t n, int C, int N, const float* dt_bias, const float* A2, const float* D, float* state, void* y,
                        int64_t ldy, void* stream);
/* One token of it; dbc = [R step inputs, B, C], the step projection w_dt [C, ldw] (type dt) is applied here. */
int scmx_scan_step(const float* x, const float* z, const float* dbc, const void* w_dt, int64_t ldw, int dt, int C, int N, int R,
                   const float* dt_bias, const float* A2, const float* D, float* state, float* y, void* stream);

/* Retention over n tokens, S <- decay_h S + k v^T, o = S^T q (o float32 [n, H, dv]); state [H, d, dv] is carried.  q and k are
 * rotated on their first `dims` elements by the rows of cs [n, dims] (cos, then sin), k is multiplied by kscale.
 * scratch NULL: token by token on the CUDA cores, any sizes.  Otherwise the chunk-parallel tensor-core form (bfloat16, positive
 * decays) with scmx_retention_scratch bytes, 256-byte aligned; 0 bytes: the sizes have no such form.  status: int32[4]. */
int64_t scmx_retention_scratch(int64_t n, int H, int d, int dv, int dims, int64_t ldv);
int scmx_retention(const void* q, int64_t ldq, const void* k, int64_t ldk, const void* v, int64_t ldv, int dt, int64_t n, int H, int d, int dv,
                   const float* cs, int dims, float kscale, const float* decay, float* state, float* o, void* scratch, int64_t scratch_bytes,
                   int32_t* status, void* stream);
/* One token of it with head norm and gate: y = o / rms(o) silu(g).  cs is the whole table; its row is the position. */
int scmx_retention_step(const float* q, const float* k, const float* v, const float* g, int H, int d, int dv, const float* cs, int64_t cs_rows,
                        int dims, int64_t pos, const int32_t* pos_dev, float kscale, const float* decay, float eps, float* state, float* y,
                        void* stream);

/* Gated delta rule over n tokens: S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q (o float32 [n, H, dv]); state [H, d, dv]
 * is carried.  q, k [n, G d] and v [n, H dv] are made here into unit vectors (q also times d^(-1/2)); head h uses q / k head
 * h / (H / G).  b [n, H]: logits of beta.  log g = nA_h softplus(a + dt_bias): channel 0: a [n, H] in storage type, dt_bias [H];
 * channel 1: a float32 [n, H d], dt_bias [H d], a decay per row of S.  d <= 256.
 * scratch NULL: token by token, any types.  Otherwise the chunk-parallel tensor-core form (bfloat16) with scmx_delta_scratch
 * bytes, 256-byte aligned; 0 bytes: the sizes have no such form.  status: int32[4]. */
int64_t scmx_delta_scratch(int64_t n, int H, int d, int dv, int64_t ldv);
int scmx_delta(const void* q, int64_t ldq, const void* k, int64_t ldk, const void* v, int64_t ldv, const void* b, int64_t ldb, const void* a,
               int64_t lda, int dt, int channel, int64_t n, int H, int G, int d, int dv, const float* nA, const float* dt_bias, float* state,
               float* o, void* scratch, int64_t scratch_bytes, int32_t* status, void* stream);
/* One token of it with head norm and gate, y = o / rms(o) w gate.  wa, wg NULL: a decay per head from the logits a [H], gate =
 * silu(g [H dv]).  Otherwise a [ra] and g [rg] are low-rank vectors: decay logits wa [H d, lwa] a, gate = sigmoid(wg [H dv, lwg] g);
 * the weights have type dt and zero padded rows of a multiple of 8 columns. */
int scmx_delta_step(const float* q, const float* k, const float* v, const float* b, const float* a, const float* g, const void* wa, int64_t lwa,
                    int ra, const void* wg, int64_t lwg, int rg, int dt, int H, int G, int d, int dv, const float* nA, const float* dt_bias,
                    const float* w, float eps, float* state, float* y, void* stream);

/* Latent attention.  A cache row holds c (R values, zero padded to a multiple of 8) and the rotated key part (r values, padded
 * likewise); the padding must be zero.  cs [cs_rows, r]: cos, then sin per position, for pairs of neighbouring elements.
 * window 0: all positions; otherwise position i sees the last `window` up to itself.
 * append: y = [query latent Q, latent R, key part r] per row -> cq [n, Q] = normalized, cache rows pos .. */
int scmx_latent_append(const void* y, int64_t ldy, int in_dt, int cache_dt, int q_dt, int64_t n, int Q, int R, int r, const float* qw,
                       const float* cw, const float* cs, int64_t cs_rows, float eps, int64_t pos, const int32_t* pos_dev, void* cq,
                       int64_t ldcq, void* cache, int64_t ldc, int64_t cap, void* stream);
/* In place: the last r elements of every head of q [n, H (d + r)]; cs: the rows of these positions. */
int scmx_latent_rotate(void* q, int64_t ldq, int dt, const float* cs, int64_t n, int H, int d, int r, void* stream);
/* out float32 [n, H, R + r] = [W_uk,h^T q_h, rotated part]; wuk [H d, ldw]. */
int scmx_latent_absorb(const void* q, int64_t ldq, int q_dt, const void* wuk, int64_t ldw, int w_dt, const float* cs, int64_t cs_rows, int64_t n,
                       int H, int d, int R, int r, int64_t pos, const int32_t* pos_dev, float* out, void* stream);
/* Softmax attention of absorbed queries (rows at pos, pos + 1, ..) over the cached latents, positions cut into nsplit <= 64
 * ranges: part float [n, H, nsplit, R rounded up to 4, + 4] for scmx_latent_value with the same pos, cap, window and nsplit.  R <= 1024. */
int scmx_latent_rows(const float* q, const void* cache, int64_t ldc, int dt, int64_t n, int64_t pos, const int32_t* pos_dev, int64_t cap,
                     int64_t window, int H, int R, int r, float scale, int nsplit, float* part, void* stream);
/* out [n, H dv] = W_uv,h (combined latent); wuv [H dv, ldw]. */
int scmx_latent_value(const float* part, const void* wuv, int64_t ldw, int w_dt, int64_t n, int64_t pos, const int32_t* pos_dev, int64_t cap,
                      int64_t window, int H, int R, int dv, int nsplit, void* out, int64_t ldo, int out_dt, void* stream);
/* The same for prompt portions on tensor cores, from per-head keys and values: q bfloat16 [n, H (d + r)] with rotated parts, kv
 * [pos + n - k0, ldkv] = per position k0 .. all heads' keys (H d), then values (H dv); rot: the rotated key parts of the same
 * positions.  k0 is not beyond the first position that row 0 sees.  Sizes: d, dv <= 128, r <= 64, multiples of 8; scale > 0. */
int scmx_latent_attn(const void* q, int64_t ldq, const void* kv, int64_t ldkv, const void* rot, int64_t ldrot, int64_t n, int64_t pos, int64_t k0,
                     int64_t window, int H, int d, int r, int dv, float scale, void* o, int32_t* status, void* stream);

/* RMS norm of q (2 H vectors of d) and k (2 G vectors) with weights qw, kw; q -> q_out [2 H, n, d], k and v appended to the caches
 * [2 G, cap, d] and [G, cap, dv] at row pos. */
int scmx_qk_norm_append(const void* q, int64_t ldq, const void* k, int64_t ldk, const void* v, int64_t ldv, int in_dt, int cache_dt, int q_dt,
                        int64_t n, int H, int G, int d, int dv, const float* qw, const float* kw, float eps, int64_t pos,
                        const int32_t* pos_dev, void* q_out, void* k_cache, void* v_cache, int64_t cap, void* stream);
/* Differential attention of n rows at positions pos .. pos+n-1 over the cache: per head o = a1 - lambda a2, o / rms(o) (1 - diff).
 * form: 0 = choose, 1 = CUDA cores (any sizes), 2 = tensor cores (bfloat16, sizes up to 128, multiples of 8; status: int32[4]). */
int scmx_diff_attn(const void* q, const void* k_cache, const void* v_cache, int dt, int64_t n, int64_t pos, int64_t cap, int H, int G, int d,
                   int dv, float scale, float lambda, float diff, float eps, void* o, int form, int32_t* status, void* stream);
/* One row of it; part f32 [G, nsplit, 2 H / G, dv + 2], counters int32 [H] (zero before the first call, left at zero), nsplit <= 32. */
int scmx_diff_decode(const float* q, const void* k_cache, const void* v_cache, int dt, int64_t n_pos, const int32_t* pos_dev, int64_t cap,
                     int H, int G, int d, int dv, float scale, float lambda, float diff, float eps, int nsplit, float* part,
                     int32_t* counters, float* o, void* stream);

/* out [M, N] = A [M, K] . W [N, K]^T, bfloat16 operands, float32 accumulation; act 1: xIELU with a_pos = softplus(p) and
 * a_neg = 1/2 + softplus(q); act 2: gelu(gate) up of columns that alternate 16 gate and 16 up (N / 2 outputs).  The pitches are multiples of 8; the output pitch covers N rounded up to 16 bytes (the padding is
 * written).  tile: 0 = choose, 64 / 128 = one CTA per 128 x tile, 256 = CTA pairs.  splits > 1: K is cut
 * into that many ranges computed side by side (no activation; part: float [splits][M][N rounded up to 4]), for products with few
 * output tiles.  status: int32[4]. */
int scmx_gemm_bf16(const void* A, int64_t lda, const void* W, int64_t ldw, int64_t M, int64_t N, int64_t K, int act, float a_pos, float a_neg,
                   void* out, int out_f32, int64_t ldo, int tile, int splits, float* part, int32_t* status, void* stream);
/* out [N] = W [N, K] x.  epi 0: plain; 1: xIELU; 2: the first C rows pass the causal convolution + SiLU of scmx_conv_silu;
 * 3: gelu(gate) up of rows that alternate 16 gate and 16 up (N / 2 outputs).
 * Rows of W are zero padded to a multiple of 8 columns. */
int scmx_gemv_x(const void* W, int64_t ldw, int dt, const float* x, int64_t N, int64_t K, int epi, float a_pos, float a_neg,
                const float* conv_w, const float* conv_b, float* tail, int C, int taps, float* out, void* stream);

#ifdef __cplusplus
}
#endif
#endif
