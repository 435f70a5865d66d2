/*
 * tpx_b200 — C ABI of the hybrid decoders' mechanisms: a linear with row strides, 32-bit or bf16 operands and 32-bit
 * results; the post-norm residual sum with its input convolution; latent attention over a windowed page cache; the
 * generalized delta rule; the Dynamic Tanh stream; gated linear attention; chunked differential attention. Conventions are those of tpx_b200.h. `f32` fields select the activation type of a call: 0 =
 * bf16 tensors, 1 = fp32 tensors (all arithmetic in true 32-bit). The residual stream, norms, gates, rotation angles,
 * scores and recurrent state are 32-bit in both.
 *
 * Sequences of a batch are padded on the left: `start[b]` tokens of sequence b are padding (NULL: none). A token's index
 * counts the padding, its position does not. `past` tokens are cached before the call; when dev_len is set the count is
 * read on the device instead (CUDA-graph decoding, one token per call).
 */
#ifndef TPX_HYBRID_H
#define TPX_HYBRID_H

#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

/* further activations of tpx_linear: tanh; xIELU with act_params = {softplus(p), 1/2 + softplus(q)}:
 * z > 0: a0 z^2 + z/2, else a1 (e^z - 1 - z) + z/2 */
enum { TPX_ACT_TANH = 4, TPX_ACT_XIELU = 5, TPX_ACT_CLAMPED_GLU = 6 };

/* y[M][N] = act(x[M][K] . w[N][K]^T + bias[N]); the activation applies to columns n >= act_from. Leading dimensions in
 * elements. bf16 operands run on the tcgen05 kernel and need K, ldx, ldw multiples of 8 and 16-byte aligned bases; fp32
 * operands run on the 32-bit kernel and need nothing. scratch as tpx_linear_bf16_tc.
 *
 * TPX_ACT_CLAMPED_GLU: the columns from act_from (even) on are pairs (g, u) of one gated unit each, which gives
 * z[M][(N - act_from) / 2] = g' s(1.702 g') (u' + 1) with s the logistic function, g' = min(g, limit) and u' clamped to
 * +-limit; y has the columns before act_from only.
 *
 * x_out != NULL: the result is added to a residual stream and normed for its next reader, nothing goes to y:
 * x_out = res + result + add (fp32 rows of ldr; add [N] may be NULL), h = tanh(norm_alpha x_out) norm_w + norm_b. */
typedef struct {
  const void *w, *x;
  const float *bias, *act_params; /* NULL: none */
  void* y;
  int64_t M, N, K, ldw, ldx, ldy;
  int f32, out_f32, act, act_from;
  void* scratch;
  size_t scratch_bytes;
  void* z;
  const float *res, *add, *norm_w, *norm_b;
  float* x_out;
  void* h;
  int64_t ldz, ldr, ldh;
  float limit, norm_alpha;
} TpxLinear;
int tpx_linear(const TpxLinear* a, void* stream);

/* One sub-layer boundary: x_out = norm(alpha * x + y) * (1 + w) with an RMS norm, then h = x_out + conv(x_out), a causal
 * per-channel convolution over time whose last taps - 1 inputs live in state[B][taps-1][D] (oldest first, updated in
 * place). With ids != NULL the stream starts here: x_out = embed[ids]. conv == NULL: no convolution and no h. Padding rows
 * become zero. conv is [taps][D]. h rows have ldh elements, columns D..ldh-1 are set to zero. */
typedef struct {
  const int64_t* ids;
  const void* embed;
  const float *x, *y, *w, *conv;
  float* state;
  const int32_t *start, *dev_len;
  float* x_out;
  void* h;
  int64_t B, S, D, ldh, past;
  float alpha, eps;
  int taps, f32;
} TpxPostnormConv;
int tpx_postnorm_conv(const TpxPostnormConv* a, void* stream);

/* The end of the stream for rows[n] (indices into the token rows): norm(norm(alpha * x + y) * (1 + w)) * (1 + w_final). */
typedef struct {
  const float *x, *y, *w, *w_final;
  const int64_t* rows;
  void* out;
  int64_t n, D, ldo;
  float alpha, eps;
  int f32;
} TpxPostnormFinal;
int tpx_postnorm_final(const TpxPostnormFinal* a, void* stream);

/* Greedy pick over fp32 logits [rows][n], first of equal maxima. */
int tpx_argmax_f32(const float* x, int64_t rows, int64_t n, int64_t* out, void* stream);

/* Rows of the latent cache: R elements = kv_rank latent values, zeros up to `krp`, rot_dim rotated key values, zeros up to
 * R. With krp and the rotated part padded to multiples of 16 and R 8 more than their sum, the tensor-core decode serves. The cache is `npages` pages of [B][32][R]; token t lives in page (t / 32) mod npages, so that a windowed layer reuses
 * its pages. A call with several tokens also has them in `lat` [B][L][R], whose row i holds token past - (L - S) + i. */
typedef struct {
  const float* proj; /* [T][ldp] fp32: q_rank query latents, then (own_kv) kv_rank + rot_dim, then heads gate inputs */
  const float *q_norm, *kv_norm;
  const double* freq; /* [rot_dim / 2] */
  const int32_t *start, *dev_len;
  void* cq;       /* [T][ldq], zero beyond q_rank */
  float* cos_sin; /* [T][rot_dim / 2][2] */
  float* gate;    /* [T][heads] sigmoid of the gate inputs */
  void* lat;      /* NULL: pages only */
  const uint64_t* pages;
  int64_t B, S, L, ldp, ldq, past, npages, q_rank, kv_rank, krp, rot_dim, R, heads;
  float eps;
  int own_kv, f32;
} TpxLatentPrep;
int tpx_latent_prep(const TpxLatentPrep* a, void* stream);

/* The cached tokens past - n .. past - 1 into rows 0 .. n-1 of lat [B][L][R]. */
int tpx_latent_gather(const uint64_t* pages, int64_t npages, int64_t B, int64_t R, int64_t past, int64_t n, int64_t L, void* lat,
                      int f32, void* stream);

/* Queries in the latent space: qa[T][heads][R] = (W_uk(head)^T q_plain, rotated q_rot), from q[T][ldq] laid out head by head
 * as (dim, rot_dim); w_uk [heads * dim][krp]. */
typedef struct {
  const void *q, *w_uk;
  const float* cos_sin;
  void* qa;
  int64_t T, ldq, heads, dim, kv_rank, krp, rot_dim, R;
  int f32;
} TpxLatentAbsorb;
int tpx_latent_absorb(const TpxLatentAbsorb* a, void* stream);

/* Softmax attention in the latent space: ol[T][heads][krp] = sum_j p_j c_j over the keys j of the token's window
 * (window tokens including itself), from the pages (lat == NULL, S == 1) or from lat [B][L][R]. */
/* The copies of the bf16 single-token kernel are waited for with a bound: tpx_latent_decode_status reads (and clears) the
 * code of a wait that gave up. */
typedef struct {
  const void *qa, *lat;
  const uint64_t* pages;
  const int32_t *start, *dev_len;
  void* ol;
  int64_t B, S, L, past, npages, heads, krp, R, window;
  float scale;
  int f32;
} TpxLatentAttn;
int tpx_latent_attn(const TpxLatentAttn* a, void* stream);
int tpx_latent_decode_status(void* stream, unsigned* status_host);

/* out[T][ldo] = gate * (W_uv(head) ol), head by head; w_uv [heads * vdim][krp]; columns beyond heads * vdim set to zero. */
typedef struct {
  const void* ol;
  const float* gate;
  const void* w_uv;
  void* out;
  int64_t T, heads, vdim, krp, ldo;
  int f32;
} TpxLatentValue;
int tpx_latent_value(const TpxLatentValue* a, void* stream);

/* Several bf16 tokens at once with keys and values expanded from the latents: out[T][ldo] = gate * softmax attention, window
 * and keys as in tpx_latent_attn. kv [B * L][ldkv] holds, per row of lat, heads * dim keys and then heads * vdim values; q
 * [T][ldq] is rotated in place. Runs on tcgen05; tpx_latent_prefill_serves says for which head sizes. The waits inside are
 * bounded: tpx_latent_tc_status reads (and clears) the code of one that gave up. */
typedef struct {
  void* q;
  const void *kv, *lat;
  const float *cos_sin, *gate;
  const int32_t* start;
  void* out;
  int64_t B, S, L, past, heads, dim, rot_dim, vdim, krp, R, ldq, ldkv, ldo, window;
  float scale;
} TpxLatentPrefill;
int tpx_latent_prefill_serves(int64_t dim, int64_t rot_dim, int64_t vdim);
int tpx_latent_prefill(const TpxLatentPrefill* a, void* stream);
int tpx_latent_tc_status(void* stream, unsigned* status_host);

/* Generalized delta rule over S tokens: per head and token, with u = k / sqrt(sum k^2 + 1e-6), decay w = exp(-e^(-1/2)
 * sigmoid(wraw)), rate a = sigmoid(araw + a_bias):  S <- diag(w) S - (a u)(u^T S) + k v^T,  o = S^T r; then o over its root
 * mean square, times norm_w, times sigmoid(g). proj [T][ldp] holds r, k, v, araw, g (heads * dim columns each); state
 * [B][heads][dim][dim] fp32 is updated in place; raw [T][heads * dim] fp32 is working space; out rows have ldo elements. */
typedef struct {
  const void* proj;
  const float *wraw, *a_bias, *norm_w;
  const int32_t *start, *dev_len;
  float *state, *raw;
  void* out;
  int64_t B, S, past, ldp, ldo, heads, dim;
  float eps;
  int f32;
} TpxDeltaRule;
int tpx_delta_rule(const TpxDeltaRule* a, void* stream);

/* The residual stream at its start, or between two layers without a linear in front: x_out[n][D] = scale embed[ids] (ids !=
 * NULL) or x, plus add [D] (may be NULL); h[n][ldh] = tanh(alpha x_out) w + b, columns from D on zero. x_out may be NULL. */
typedef struct {
  const int64_t* ids;
  const void* embed; /* [vocab][D] */
  const float *x, *add, *w, *b;
  float* x_out;
  void* h;
  int64_t n, D, ldh;
  float scale, alpha;
  int f32;
} TpxDyt;
int tpx_dyt(const TpxDyt* a, void* stream);

/* Gated linear attention over S tokens: per head and token S <- diag(w) S + k v^T, o = S^T (q / sqrt(dim)), with the decay
 * w = s(z)^(1/tau) per key channel, s the logistic function; then o over its root mean square, times norm_w [vdim], times
 * g s(g). proj [T][ldp] holds q and k (heads * dim columns each), v and g (heads * vdim each) from the columns given on. z is
 * read from zraw [T][heads * dim], or, for a single token that tpx_gla_token_serves, computed as a2 [heads * dim][lda2] times
 * the `rank` columns of proj from a1_col on, plus a2_bias (zraw == NULL). state [B][heads][dim][vdim] fp32 is updated in
 * place; raw [T][heads * vdim] fp32 is working space; out rows have ldo elements. Padding rows of out become zero. */
typedef struct {
  const void* proj;
  const float* zraw;
  const void* a2;
  const float *a2_bias, *norm_w;
  const int32_t *start, *dev_len;
  float *state, *raw;
  void* out;
  int64_t B, S, past, ldp, ldo, lda2, rank, heads, dim, vdim, q_col, k_col, v_col, g_col, a1_col;
  float tau, eps;
  int f32;
} TpxGla;
int tpx_gla_token_serves(int64_t dim, int64_t vdim);
int tpx_gla(const TpxGla* a, void* stream);

/* Chunked differential attention with capped scores. proj [T][ldp] holds heads x (2 x dim) queries, kv_heads x (2 x dim) keys
 * and kv_heads x vdim values from the columns given on. A token at position i (leading padding not counted) sees the tokens of
 * its chunk, positions i / chunk * chunk .. i. Per map m: softmax of softcap tanh(scale q_m . k_m / softcap); with the maps'
 * outputs a1 and a2, o = a1 - lambda a2, then o over its root mean square, times `mult`. Query head h reads key / value head
 * h / (heads / kv_heads).
 *
 * The cache is `npages` pages of [B][kv_heads][32][R]: token t in page (t / 32) mod npages; a row holds map 1's key, map 2's key
 * (each padded with zeros to dp = dim rounded up to 16), the value, and zeros up to R, which is 2 dp + vdim rounded up to 16, plus 8.
 * The call appends its tokens. Several tokens also need the earlier rows that are still in reach: back = min(past, chunk - 1) of
 * them (L = back + S); `live` [B][L][kv_heads][R] is working space for them and the new rows, which may be NULL when back is 0
 * and tpx_diff_prefill_serves. The waits inside the bf16 kernels are bounded: tpx_diff_status reads (and clears) the code of
 * one that gave up. */
typedef struct {
  const void* proj;
  const uint64_t* pages;
  void* live;
  const int32_t *start, *dev_len;
  void* out;
  int64_t B, S, L, past, npages, ldp, ldo, heads, kv_heads, dim, vdim, R, chunk, q_col, k_col, v_col;
  float scale, softcap, lambda, mult, eps;
  int f32;
} TpxDiffAttn;
int tpx_diff_prefill_serves(int64_t dim, int64_t vdim, float softcap);
int tpx_diff_attn(const TpxDiffAttn* a, void* stream);
int tpx_diff_status(void* stream, unsigned* status_host);

#ifdef __cplusplus
}
#endif
#endif /* TPX_HYBRID_H */
