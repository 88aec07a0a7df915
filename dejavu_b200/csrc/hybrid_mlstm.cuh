// Arguments and device helpers shared by the mLSTM kernels.
#pragma once
#include "mma.cuh"

namespace djv {

constexpr int ML_THREADS = 256;

struct MlstmArgs {
  void *out;
  const void *proj;      // rows of q (H, dk) | k (H, dk) | v (H, dv) | output gate (H, dv)
  long long ld;
  const float *gates;    // rows of input gate (H) | forget gate (H), before bias and cap
  long long ldg;
  const float *bias_i, *bias_f;
  float cap;
  const float *norm;     // (H, dv)
  float eps, scale;
  float *state;          // (B, H, mlstm_state_stride)
  const long long *pos;
  int B, n, H, dk, dv;
  int C, nc;             // chunk length, number of chunks
  float *contrib;        // (B, H, nc, dk * dv + dk): a chunk's own S and n, then the incoming ones
  double *chunk;         // (B, H, nc, 3): sum of log f, maximum of a, incoming m
  bf16 *s_hi, *s_lo;     // (B, H, nc, dk, dv): incoming S as two bf16 terms (tensor-core form)
  float2 *g_a;           // (B, H, nc, C): a_s of every token, and (below) M_t without m_in and F_t (tensor-core form)
  double *g_run, *g_sum;
};

// a head's state: S (dk, dv), n (dk), m
__host__ __device__ __forceinline__ int mlstm_state_stride(int dk, int dv) { return (dk * dv + dk + 1 + 3) & ~3; }
__host__ __device__ __forceinline__ size_t mlstm_contrib_stride(int dk, int dv) { return (size_t)((dk * dv + dk + 3) & ~3); }

__device__ __forceinline__ float softcap_f(float z, float cap) { return cap * tanhf(z / cap); }

// An exponent that is a difference of sums: two floats, hi + lo, keep what one would lose when the sums are large.
__device__ __forceinline__ float2 split_double(double v) {
  const float hi = (float)v;
  return make_float2(hi, isinf(hi) ? 0.f : (float)(v - (double)hi));
}
// exp(a - m) of such pairs
__device__ __forceinline__ float exp_diff(float2 a, float2 m) { return expf((a.x - m.x) + (a.y - m.y)); }

// The gates of a chunk of cl <= 32 * PER tokens, by one warp. With F_t the sum of log f over the chunk up to and
// including t, token s weighs exp(a_s - M_t) at token t, a_s = log i_s - F_s, M_t = max(m_in, a_0 .. a_t), and
// m_t = F_t + M_t. Tokens past the end: a = -inf, log f = 0.
// a_s: pairs; run (may be null): M_t with m_in = -inf, as doubles; fsum: F_t (may be null).
template <int PER>
__device__ __forceinline__ void chunk_gates(const MlstmArgs &a, int b, int h, int t0, int cl, float2 *a_s, double *run,
                                            double *fsum, double &f_total, double &a_max) {
  const int lane = threadIdx.x % WARP;
  const float bi = a.bias_i[h], bf = a.bias_f[h];
  const float *g = a.gates + ((size_t)b * a.n + t0) * a.ldg + h;
  double f[PER], v[PER];
  float zi[PER], zf[PER];
#pragma unroll
  for (int x = 0; x < PER; ++x) {
    const int t = lane * PER + x;
    zi[x] = t < cl ? g[(size_t)t * a.ldg] : 0.f;
    zf[x] = t < cl ? g[(size_t)t * a.ldg + a.H] : 0.f;
  }
#pragma unroll
  for (int x = 0; x < PER; ++x) {
    const int t = lane * PER + x;
    f[x] = t < cl ? (double)log_sigmoid_f(softcap_f(zf[x] + bf, a.cap)) : 0.0;
    v[x] = t < cl ? (double)softcap_f(zi[x] + bi, a.cap) : -INFINITY;
    if (x) f[x] += f[x - 1];
  }
  double sum = f[PER - 1];
#pragma unroll
  for (int o = 1; o < WARP; o <<= 1) {
    const double up = __shfl_up_sync(0xffffffffu, sum, o);
    if (lane >= o) sum += up;
  }
  const double before = sum - f[PER - 1];
  f_total = __shfl_sync(0xffffffffu, sum, WARP - 1);
  double m[PER];
#pragma unroll
  for (int x = 0; x < PER; ++x) {
    f[x] += before;
    v[x] -= f[x];
    m[x] = x ? fmax(m[x - 1], v[x]) : v[x];
  }
  double top = m[PER - 1];
#pragma unroll
  for (int o = 1; o < WARP; o <<= 1) {
    const double up = __shfl_up_sync(0xffffffffu, top, o);
    if (lane >= o) top = fmax(top, up);
  }
  a_max = __shfl_sync(0xffffffffu, top, WARP - 1);
  double prev = __shfl_up_sync(0xffffffffu, top, 1);
  if (lane == 0) prev = -INFINITY;
#pragma unroll
  for (int x = 0; x < PER; ++x) {
    const int t = lane * PER + x;
    a_s[t] = split_double(v[x]);
    if (run) run[t] = fmax(m[x], prev);
    if (fsum) fsum[t] = f[x];
  }
}

// tensor-core form of the chunk kernels (bf16); chunks of MLSTM_TC_CHUNK tokens
constexpr int MLSTM_TC_CHUNK = 128;
bool mlstm_tc_supported(int dtype, int dk, int dv);
int mlstm_tc_gates(const MlstmArgs &a, cudaStream_t st);
int mlstm_tc_chunk_state(const MlstmArgs &a, cudaStream_t st);
int mlstm_tc_chunk_out(const MlstmArgs &a, cudaStream_t st);

}  // namespace djv
