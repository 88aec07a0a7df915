/*
 * dejavu_b200_routed.h — C ABI of the kernels for decoders that mix matrix memories (mLSTM), windowed latent attention and
 * routed feed-forwards (libdejavu_b200_routed.so, which also has the functions marked (both) in dejavu_b200_hybrid.h).
 *
 * Conventions as in dejavu_b200_hybrid.h: T is the element type of weights and activations (bf16 or fp32); norm weights,
 * gates, states, scores, router logits and sums are fp32 whatever T is; rows are ordered (sequence, token); `pos` holds B
 * int64 on the device.
 */
#ifndef DEJAVU_B200_ROUTED_H
#define DEJAVU_B200_ROUTED_H

#include "dejavu_b200_hybrid.h"

#ifdef __cplusplus
extern "C" {
#endif

/* Matrix memory. proj rows hold q (H, dk) | k (H, dk) | v (H, dv) | output gate (H, dv); gates rows hold the input (H) and
 * forget (H) gates' projections, fp32. With i = cap tanh((z_i + bias_i) / cap), f = log_sigmoid(cap tanh((z_f + bias_f) / cap))
 *   m' = max(f + m, i);  S' = e^(f + m - m') S + e^(i - m') k v^T;  n' = e^(f + m - m') n + e^(i - m') k
 *   o = S'^T (q scale) / (max(|n' . (q scale)|, e^(-m')) + 1e-6);  out = o / rms(o) * norm * sigmoid(output gate)
 * norm (H, dv). state (B, H, djv_mlstm_state_floats) fp32: S (dk, dv), n (dk), m; read and written; a sequence whose pos
 * is 0 starts from zero whatever it holds. djv_mlstm_prefill takes n tokens per sequence in chunks that run in parallel;
 * djv_mlstm_decode takes one, whose projections are fp32 (out is T). */
int djv_mlstm_state_floats(int dk, int dv);
size_t djv_mlstm_scratch_bytes(int dtype, int B, int n, int H, int dk, int dv);
int djv_mlstm_prefill(int dtype, void *out, const void *proj, long long ld, const float *gates, long long ldg,
                      const float *bias_i, const float *bias_f, float cap, const float *norm, float eps, float scale,
                      float *state, const long long *pos, int B, int n, int H, int dk, int dv, void *scratch,
                      size_t scratch_bytes, void *stream);
int djv_mlstm_decode(int dtype, void *out, const float *proj, long long ld, const float *gates, long long ldg,
                     const float *bias_i, const float *bias_f, float cap, const float *norm, float eps, float scale,
                     float *state, const long long *pos, int B, int H, int dk, int dv, void *stream);
/* Waits of the tensor-core chunk kernels on their own products that ran out since load (0 in a healthy process). */
unsigned djv_mlstm_timeouts(void);

/* Latent attention. A token's cache row is its RMS-normed latent (rank) and a rotated key part (rot, pairs (2i, 2i + 1))
 * that all heads share; the ring (B, cap, rank + rot) holds position p in slot p % cap, cap >= min(window, longest sequence).
 * djv_latent_rows, store = 0: rows (B, past + n, rank + rot) from the ring (positions pos - past .. pos - 1, zeros before
 * position 0) and from proj (B*n rows of latent | key part, ld apart). store = 1: the last min(n, cap) of these rows enter
 * the ring (proj is not read); store = 2: both, for past = 0. `past` is no less than what a sequence can see of its earlier tokens. */
int djv_latent_rows(int dtype, void *rows, const void *proj, long long ld, void *ring, const float *norm, float eps,
                    const float *freqs, const long long *pos, int B, int n, int past, int rank, int rot, int cap,
                    int store, void *stream);
/* Causal attention of n new tokens per sequence. q (B*n) rows of (H, dim + rot), rotated; kv (B * (past + n)) rows of
 * k (H, dim) | v (H, dv); tail: rows as kv whose first `rot` elements are the shared key part. Position i sees j with
 * 0 <= i - j < window. out (B*n, H*dv) of T, times sigmoid(gate) if gate (rows of (H, dv)) is given. */
int djv_latent_attn(int dtype, void *out, const void *q, long long ldq, const void *kv, long long ldkv, const void *tail,
                    long long ldt, const void *gate, long long ldg, const long long *pos, int B, int n, int past, int H,
                    int dim, int rot, int dv, int window, float scale, void *stream);
/* The decode step of the same on the ring itself. proj rows hold q (H, dim + rot) | latent (rank) | key part (rot), neither
 * normed nor rotated; uk (H*dim, rank), uv (H*dv, rank). stages is a sum of
 *   1  qc (B, H, rank + rot) = (uk_h^T q_h | rotated q_h), and the token's row enters the ring
 *   2  scratch (djv_latent_scratch_floats with window <= cap) = weighted sums of the rows' latents over parts of the window,
 *      weights from softmax(qc . ring rows * scale)
 *   4  out (B, H*dv) = uv_h applied to the parts put together, times sigmoid(gate) */
size_t djv_latent_scratch_floats(int B, int H, int rank, int window);
int djv_latent_decode(int dtype, void *out, void *qc, float *scratch, size_t scratch_floats, const void *proj, long long ld,
                      const void *uk, const void *uv, const float *norm, float eps, const float *freqs, void *ring,
                      const void *gate, long long ldg, const long long *pos, int B, int H, int dim, int rot, int dv,
                      int rank, int cap, int window, float scale, int stages, void *stream);

/* Routed feed-forward: a token's `top` largest router logits z choose its experts, with weights sigmoid(z).
 * djv_moe_route sorts n tokens' choices by expert: xs (n*top, D) their activations, ws (n*top) their weights, offsets
 * (E + 1) every expert's first row, place (n, top) the row of each choice. expert, weight (n, top) and count (E): scratch. */
int djv_moe_route(int dtype, void *xs, const void *x, const float *z, int *expert, int *place, float *weight, float *ws,
                  int *count, int *offsets, int n, int E, int top, int D, void *stream);
/* y = (scale * x) w_e^T over the rows of each expert e: x (R, K), w (E, N, K), y (R, N) of T; glu: rows 2i, 2i + 1 of an
 * expert are gate and up, y (R, N / 2) = silu(gate) * up. scale (R) or NULL. */
int djv_moe_grouped(int dtype, void *y, const void *x, const void *w, const float *scale, const int *offsets, int R, int E,
                    int N, int K, int glu, void *stream);
/* The decode step's feed-forward of B rows: y (B, D) fp32 = init + sum of the chosen experts' outputs (+ the shared one's).
 * w_gu (E, 2F, D), w_down (E, D, F); shared_gu (2F', D) and shared_down (D, F') or NULL. act (B, top + shared, ld_act) of
 * T and chosen (B, top): scratch. stages: 1 the gated units, 2 the down products, 3 both. */
int djv_moe_decode(int dtype, float *y, void *act, int *chosen, const void *x, const float *z, const void *w_gu,
                   const void *w_down, const void *shared_gu, const void *shared_down, const float *init, int B, int E,
                   int top, int D, int F, int F_shared, int ld_act, int stages, void *stream);
/* Waits of the tensor-core grouped product that ran out since load (0 in a healthy process). */
unsigned djv_moe_timeouts(void);

#ifdef __cplusplus
}
#endif
#endif /* DEJAVU_B200_ROUTED_H */
