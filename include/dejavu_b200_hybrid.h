/*
 * dejavu_b200_hybrid.h — C ABI of the kernels for decoders that mix gated linear attention, sliding-window attention
 * with sinks, gated MLPs and hyper-connected residual streams (libdejavu_b200_hybrid.so).
 *
 * Functions marked (both) are also in libdejavu_b200_routed.so (dejavu_b200_routed.h).
 *
 * Same conventions as dejavu_b200.h: raw device pointers, sizes, a CUDA stream as void*; work is only enqueued, never
 * allocated; DJV_OK or a negative DJV_ERR_* with a message in djv_last_error() (each library has its own). `dtype` is
 * the element type T of weights and activations (DJV_DTYPE_BF16 or DJV_DTYPE_F32); residual streams, norm weights,
 * decays, states, scores and logits are fp32 whatever T is.
 *
 * Rows of activations are ordered (sequence, token): row = b * n + t for B sequences of n tokens each. `pos` points to
 * B int64 on the device: the position of each sequence's first token of the call. Positions live on the device so that
 * a captured CUDA graph of a step stays valid.
 */
#ifndef DEJAVU_B200_HYBRID_H
#define DEJAVU_B200_HYBRID_H

#include "dejavu_b200.h"

#ifdef __cplusplus
extern "C" {
#endif

/* (both) One boundary between sublayers of a decoder whose residual is S parallel streams (1 <= S <= 8), in one pass:
 *   new_t = sum_s mix[s*S + t] * x_s + w_out[t] * y        (y = NULL: new = x)
 *   u     = sum_t w_in[t] * new_t                          (w_in = NULL: plain sum)
 *   h     = u / sqrt(mean(u^2) + eps) * gamma              (gamma = NULL: h is not written)
 * x_in (rows, S, D) fp32, or NULL: every stream starts as embed[ids[row]] (embed (vocab, D) of T, ids int64; ids out
 * of range are clamped). x_out (rows, S, D) fp32 receives new (may be x_in; NULL: not stored). y (rows, D) fp32.
 * h (R, D) of T. row_list (R int32) selects which rows are processed, NULL = rows 0..R-1. */
int djv_hyper_step(int dtype, void *h, float *x_out, const float *x_in, const float *y, const float *mix,
                   const float *w_out, const float *w_in, const float *gamma, float eps, const int32_t *row_list,
                   const long long *ids, const void *embed, int R, int S, int D, int vocab, void *stream);

/* (both) The boundary of a decoder with one residual and norms on both sides of a sublayer, in one pass:
 *   s = y + sum_k parts[part_rows[row * n_parts + k]]      (y = NULL: 0; parts = NULL: none)
 *   new = x + s / sqrt(mean(s^2) + eps) * (base + gamma_y) (gamma_y = NULL: new = x + s)
 *   h = new / sqrt(mean(new^2) + eps) * (base + gamma)     (gamma = NULL: h is not written)
 * parts: rows of D elements of T, part_rows (rows, n_parts) int32. The rest as in djv_hyper_step with S = 1. */
int djv_residual_step(int dtype, void *h, float *x_out, const float *x_in, const float *y, const void *parts,
                      const int32_t *part_rows, int n_parts, const float *gamma_y, const float *gamma, float base,
                      float eps, const int32_t *row_list, const long long *ids, const void *embed, int R, int D,
                      int vocab, void *stream);

/* (both) y[b, m] = act(w[m, :] . x[b, :]) for B <= DJV_MAX_BATCH rows of x: the decode step's matrix products. out_dtype:
 * T or DJV_DTYPE_F32. act: DJV_ACT_ID, DJV_ACT_SOFTCAP, DJV_ACT_CLAMPED_GLU, DJV_ACT_SILU_GLU (gated units: y has M/2
 * columns). */
int djv_dense_gemv(int dtype, int out_dtype, void *y, const void *w, const void *x, int B, int N, int M,
                   long long ldw, int act, float act_param, void *stream);

/* (both) y (R, F) = gated unit of gu (R, 2F), gate and up interleaved; act: DJV_ACT_CLAMPED_GLU or DJV_ACT_SILU_GLU. */
int djv_glu(int dtype, void *y, const void *gu, long long R, int F, int act, float limit, void *stream);

/* (both) y <- cap * tanh(y / cap), fp32, in place */
int djv_softcap(float *y, long long n, float cap, void *stream);

/* (both) Rotary positions in place on the first `heads` heads (dim elements apart) of every row of buf (B*n rows, ld
 * elements apart): pair i < half is dimensions (i, i + half), or (2i, 2i + 1) if interleaved; angle = position * freqs[i],
 * cos and sin times amp. */
int djv_rotary(int dtype, void *buf, long long ld, const float *freqs, float amp, const long long *pos, int B, int n,
               int heads, int dim, int half, int interleaved, void *stream);

/* Causal attention of n new tokens per sequence over themselves and the tokens the cache holds. qkv rows hold
 * q (H, dk) | k (G, dk) | v (G, dv), already rotated; H % G == 0. The caches are rings of `cap` tokens per
 * (sequence, kv head): k_ring (B, G, cap, dk), v_ring (B, G, cap, dv), position p in slot p % cap, cap >= min(window,
 * longest sequence). Position i sees j with 0 <= i - j < window. sink (H) fp32 or NULL: exp(sink_h) joins the
 * denominator. out (B*n, H*dv) of T. The caches are only read; djv_window_store afterwards writes the new tokens. */
int djv_window_attn(int dtype, void *out, const void *qkv, long long ld, const void *k_ring, const void *v_ring,
                    const float *sink, const long long *pos, int B, int n, int H, int G, int dk, int dv, int cap,
                    int window, float scale, void *stream);
int djv_window_store(int dtype, void *k_ring, void *v_ring, const void *qkv, long long ld, const long long *pos, int B,
                     int n, int H, int G, int dk, int dv, int cap, void *stream);
/* (both) Waits of the tensor-core kernels on their own products that ran out since load (0 in a healthy process; synchronises). */
unsigned djv_window_timeouts(void);
/* The decode step of the same in one kernel: rotates q and k of one token per sequence, stores k and v into the rings
 * and attends. qkv rows are not rotated yet; freqs NULL: no rotation. */
int djv_window_attn_decode(int dtype, void *out, const void *qkv, long long ld, void *k_ring, void *v_ring,
                           const float *sink, const float *freqs, float amp, int half, const long long *pos, int B,
                           int H, int G, int dk, int dv, int cap, int window, float scale, void *stream);

/* Gated linear attention. proj rows hold q (H, dk) | k (H, dk) | v (H, dv) | gate (H, dv) | t (rank); the decay of a
 * key channel is exp(log_sigmoid(a2 t + a2_bias) / tau) with a2 (H*dk, rank) fp32. Per head
 *   S <- diag(decay) S + k v^T;  o = S^T (q * scale);  out = o / rms(o) * norm * silu(gate)
 * state (B, H, dk, dv) fp32 is read and written; a sequence whose pos is 0 starts from zero whatever it holds.
 * djv_gla_prefill takes n tokens per sequence in chunks that run in parallel; djv_gla_decode takes one. */
size_t djv_gla_scratch_bytes(int dtype, int B, int n, int H, int dk, int dv);
int djv_gla_prefill(int dtype, void *out, const void *proj, long long ld, const float *a2, const float *a2_bias,
                    int rank, float inv_tau, const float *norm, float eps, float scale, float *state,
                    const long long *pos, int B, int n, int H, int dk, int dv, void *scratch, size_t scratch_bytes,
                    void *stream);
int djv_gla_decode(int dtype, void *out, const void *proj, long long ld, const float *a2, const float *a2_bias,
                   int rank, float inv_tau, const float *norm, float eps, float scale, float *state,
                   const long long *pos, int B, int H, int dk, int dv, void *stream);

#ifdef __cplusplus
}
#endif
#endif /* DEJAVU_B200_HYBRID_H */
