// Windowed attention of a prompt portion for any element type, head size and alignment, on the CUDA cores; and the choice
// between this form and the tensor-core one.
#include "../../include/dejavu_b200_hybrid.h"
#include "dtype.cuh"
#include "hybrid_attention.cuh"

namespace djv {

// A warp per (query, head): lanes take 32 keys at a time for the scores, then dv / 32 value columns each.
constexpr int WA_WARPS = 8;

template <typename T, int E>  // E * 32 >= dv
__global__ void __launch_bounds__(WA_WARPS * WARP) window_attn_simple_kernel(WindowArgs a) {
  extern __shared__ float q_sm[];  // WA_WARPS * dk
  pdl_prologue();
  const int warp = threadIdx.x / WARP, lane = threadIdx.x % WARP;
  const int t = blockIdx.x * WA_WARPS + warp, h = blockIdx.y, b = blockIdx.z;
  if (t >= a.n) return;
  const int g = h / (a.H / a.G), own = a.dk - a.rot;  // own: key dimensions of the head itself
  const long long p0 = a.pos[b], p = p0 + t, first = (long long)b * (a.past + a.n) + a.past;
  const T *qr = static_cast<const T *>(a.q) + ((size_t)b * a.n + t) * a.ldq + (size_t)h * a.dk;
  float *q = q_sm + warp * a.dk;
  for (int i = lane; i < a.dk; i += WARP) q[i] = to_f(qr[i]);
  __syncwarp();
  const bool ring = a.k_ring != nullptr;
  const T *kr = ring ? static_cast<const T *>(a.k_ring) + ((size_t)b * a.G + g) * a.cap * a.dk : nullptr;
  const T *vr = ring ? static_cast<const T *>(a.v_ring) + ((size_t)b * a.G + g) * a.cap * a.dv : nullptr;
  const T *kn = static_cast<const T *>(a.k) + first * a.ldk + (size_t)g * own;
  const T *vn = static_cast<const T *>(a.v) + first * a.ldv + (size_t)g * a.dv;
  const T *tn = a.rot ? static_cast<const T *>(a.tail) + first * a.ldt : nullptr;
  float m = a.sink ? a.sink[h] : -INFINITY, l = a.sink ? 1.f : 0.f, o[E];
#pragma unroll
  for (int e = 0; e < E; ++e) o[e] = 0.f;
  long long lo = p - a.window + 1;
  if (lo < 0) lo = 0;
  if (!ring && lo < p0 - a.past) lo = p0 - a.past;
  for (long long j0 = lo; j0 <= p; j0 += WARP) {
    const long long j = j0 + lane;
    float s = -INFINITY;
    if (j <= p) {
      s = 0.f;
      if (ring && j < p0) {
        const T *k = kr + (size_t)(j % a.cap) * a.dk;
        for (int i = 0; i < a.dk; ++i) s = fmaf(q[i], to_f(k[i]), s);
      } else {
        const T *k = kn + (j - p0) * a.ldk;
        for (int i = 0; i < own; ++i) s = fmaf(q[i], to_f(k[i]), s);
        const T *kt = tn + (j - p0) * a.ldt;
        for (int i = 0; i < a.rot; ++i) s = fmaf(q[own + i], to_f(kt[i]), s);
      }
      s *= a.scale;
    }
    const float m_new = fmaxf(m, warp_max(s));
    const float corr = m == -INFINITY ? 0.f : expf(m - m_new);
    const float w = j <= p ? expf(s - m_new) : 0.f;
    l = l * corr + warp_sum(w);
    m = m_new;
#pragma unroll
    for (int e = 0; e < E; ++e) o[e] *= corr;
    const int cnt = (int)min((long long)WARP, p - j0 + 1);
    for (int c = 0; c < cnt; ++c) {
      const float wc = __shfl_sync(0xffffffffu, w, c);
      const long long jj = j0 + c;
      const T *v = ring && jj < p0 ? vr + (size_t)(jj % a.cap) * a.dv : vn + (jj - p0) * a.ldv;
#pragma unroll
      for (int e = 0; e < E; ++e)
        if (e * WARP + lane < a.dv) o[e] = fmaf(wc, to_f(v[e * WARP + lane]), o[e]);
    }
  }
  T *out = static_cast<T *>(a.out) + (((size_t)b * a.n + t) * a.H + h) * a.dv;
  const T *gate = a.gate ? static_cast<const T *>(a.gate) + ((size_t)b * a.n + t) * a.ldg + (size_t)h * a.dv : nullptr;
#pragma unroll
  for (int e = 0; e < E; ++e) {
    const int j = e * WARP + lane;
    if (j < a.dv) out[j] = from_f<T>(o[e] / l * (gate ? sigmoid_f(to_f(gate[j])) : 1.f));
  }
}

template <typename T>
static int launch_simple(const WindowArgs &a, cudaStream_t st) {
  const dim3 grid(ceil_div(a.n, WA_WARPS), a.H, a.B);
  const size_t smem = (size_t)WA_WARPS * a.dk * 4;
#define DJV_WA(E_) djv::launch_kernel(window_attn_simple_kernel<T, E_>, grid, dim3(WA_WARPS * WARP), smem, st, a)
  if (a.dv <= 64) DJV_WA(2);
  else if (a.dv <= 128) DJV_WA(4);
  else if (a.dv <= 256) DJV_WA(8);
  else DJV_WA(16);
#undef DJV_WA
  count_launch();
  return check_launch("window_attn");
}

int window_attn_portion(int dtype, const WindowArgs &a, cudaStream_t st) {
  if (dtype == DJV_DTYPE_BF16) return window_prefill_supported(a) ? window_prefill(a, st) : launch_simple<bf16>(a, st);
  return launch_simple<float>(a, st);
}

}  // namespace djv
