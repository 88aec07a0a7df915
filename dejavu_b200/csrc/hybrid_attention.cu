// Sliding-window attention with grouped key/value heads and a learned sink per head, over ring caches that hold the
// window and nothing else.
//
//   k_ring (B, G, cap, dk), v_ring (B, G, cap, dv): position p of a sequence sits in slot p % cap.
//
// A portion of n new tokens attends over the ring (positions before the portion) and over its own keys and values,
// which are still in the projection's output; the new tokens enter the ring afterwards, because they overwrite slots
// that the portion's first tokens can still see. The decode step has one token, the slot it takes is the one that has
// just left the window, so it rotates, stores and attends in one kernel.
#include <cooperative_groups.h>

#include "../../include/dejavu_b200_hybrid.h"
#include "hybrid_attention.cuh"
#include "mma.cuh"

namespace djv {

namespace cg = cooperative_groups;

// ---- rotary positions ------------------------------------------------------------------------------------------
// One block per row; the angles of the row's position are shared by its heads.
template <typename T>
__global__ void rotary_kernel(T *__restrict__ buf, long long ld, const float *__restrict__ freqs, float amp,
                              const long long *__restrict__ pos, int n, int heads, int dim, int half) {
  extern __shared__ float cs[];  // cos[half], sin[half]
  pdl_prologue();
  const long long row = blockIdx.x;
  const int b = (int)(row / n), t = (int)(row % n);
  const float p = (float)(pos[b] + t);
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float s, c;
    sincosf(p * freqs[i], &s, &c);
    cs[i] = c * amp;
    cs[half + i] = s * amp;
  }
  __syncthreads();
  T *x = buf + row * ld;
  for (int k = threadIdx.x; k < heads * half; k += blockDim.x) {
    const int h = k / half, i = k % half;
    T *e = x + (size_t)h * dim + i;
    const float u = to_f(e[0]), v = to_f(e[half]);
    e[0] = from_f<T>(u * cs[i] - v * cs[half + i]);
    e[half] = from_f<T>(v * cs[i] + u * cs[half + i]);
  }
}

// ---- a portion of new tokens, any element type -----------------------------------------------------------------
// A warp per (query, head): lanes take 32 keys at a time for the scores, then dv / 32 value columns each.
constexpr int WA_WARPS = 8;

template <typename T, int E>  // E * 32 >= dv
__global__ void __launch_bounds__(WA_WARPS * WARP) window_attn_simple_kernel(WindowArgs a) {
  extern __shared__ float q_sm[];  // WA_WARPS * dk
  pdl_prologue();
  const int warp = threadIdx.x / WARP, lane = threadIdx.x % WARP;
  const int t = blockIdx.x * WA_WARPS + warp, h = blockIdx.y, b = blockIdx.z;
  if (t >= a.n) return;
  const int g = h / (a.H / a.G);
  const long long p0 = a.pos[b], p = p0 + t;
  const T *rows = static_cast<const T *>(a.qkv) + (size_t)b * a.n * a.ld;
  float *q = q_sm + warp * a.dk;
  for (int i = lane; i < a.dk; i += WARP) q[i] = to_f(rows[(size_t)t * a.ld + (size_t)h * a.dk + i]);
  __syncwarp();
  const T *kr = static_cast<const T *>(a.k_ring) + ((size_t)b * a.G + g) * a.cap * a.dk;
  const T *vr = static_cast<const T *>(a.v_ring) + ((size_t)b * a.G + g) * a.cap * a.dv;
  const T *kn = rows + (size_t)(a.H + g) * a.dk;
  const T *vn = rows + (size_t)(a.H + a.G) * a.dk + (size_t)g * a.dv;
  float m = a.sink ? a.sink[h] : -INFINITY, l = a.sink ? 1.f : 0.f, o[E];
#pragma unroll
  for (int e = 0; e < E; ++e) o[e] = 0.f;
  long long lo = p - a.window + 1;
  if (lo < 0) lo = 0;
  for (long long j0 = lo; j0 <= p; j0 += WARP) {
    const long long j = j0 + lane;
    float s = -INFINITY;
    if (j <= p) {
      const T *k = j < p0 ? kr + (size_t)(j % a.cap) * a.dk : kn + (size_t)(j - p0) * a.ld;
      s = 0.f;
      for (int i = 0; i < a.dk; ++i) s = fmaf(q[i], to_f(k[i]), s);
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
      const T *v = jj < p0 ? vr + (size_t)(jj % a.cap) * a.dv : vn + (size_t)(jj - p0) * a.ld;
#pragma unroll
      for (int e = 0; e < E; ++e)
        if (e * WARP + lane < a.dv) o[e] = fmaf(wc, to_f(v[e * WARP + lane]), o[e]);
    }
  }
  T *out = static_cast<T *>(a.out) + (((size_t)b * a.n + t) * a.H + h) * a.dv;
#pragma unroll
  for (int e = 0; e < E; ++e)
    if (e * WARP + lane < a.dv) out[e * WARP + lane] = from_f<T>(o[e] / l);
}

// ---- the new tokens enter the rings ----------------------------------------------------------------------------
template <typename T>
__global__ void window_store_kernel(T *__restrict__ k_ring, T *__restrict__ v_ring, const T *__restrict__ qkv,
                                    long long ld, const long long *__restrict__ pos, int n, int H, int G, int dk,
                                    int dv, int cap, int first) {
  pdl_prologue();
  const int t = first + blockIdx.x, b = blockIdx.y;  // the last min(n, cap) tokens
  const size_t slot = (size_t)((pos[b] + t) % cap);
  const T *row = qkv + ((size_t)b * n + t) * ld + (size_t)H * dk;
  for (int i = threadIdx.x; i < G * dk; i += blockDim.x)
    k_ring[(((size_t)b * G + i / dk) * cap + slot) * dk + i % dk] = row[i];
  row += (size_t)G * dk;
  for (int i = threadIdx.x; i < G * dv; i += blockDim.x)
    v_ring[(((size_t)b * G + i / dv) * cap + slot) * dv + i % dv] = row[i];
}

// ---- decode ----------------------------------------------------------------------------------------------------
// grid (G * head subgroups, B, splits); the splits of the window form a cluster, rank 0 combines them through
// distributed shared memory. A block takes RT query heads of one kv head, so K and V are read once for all of them,
// and streams tiles of up to `tile` tokens through shared memory: every load of a tile is in flight at once.
constexpr int WD_THREADS = 128;
constexpr int WD_MAX_SPLITS = 8;

struct DecodeArgs {
  WindowArgs w;
  void *k_ring, *v_ring;
  const float *freqs;
  float amp;
  int half, subs, tile, k_pitch, v_pitch, vrows;  // pitches in elements; vrows: rows of V per pass of the threads
};

// rotated element i of a head vector (fp32)
template <typename T>
__device__ __forceinline__ float rotated(const T *x, int i, const float *cs, int half) {
  const float u = to_f(x[i]);
  if (i < half) return u * cs[i] - to_f(x[i + half]) * cs[half + i];
  if (i < 2 * half) return u * cs[i - half] + to_f(x[i - half]) * cs[i];
  return u;
}

template <typename T, int RT, bool VEC>
__global__ void __launch_bounds__(WD_THREADS) window_decode_kernel(DecodeArgs d) {
  const WindowArgs &a = d.w;
  constexpr int N = VEC ? Chunk<T>::N : 1;
  extern __shared__ __align__(16) unsigned char sm_raw[];
  const int dk = a.dk, dv = a.dv, tile = d.tile;
  T *k_sm = reinterpret_cast<T *>(sm_raw);
  T *v_sm = k_sm + (size_t)tile * d.k_pitch;
  float *qs = reinterpret_cast<float *>(v_sm + (size_t)tile * d.v_pitch);  // RT * dk
  float *sc = qs + RT * dk;                                               // RT * tile
  float *cs = sc + RT * tile;                                             // 2 * half
  float *part = cs + 2 * d.half;                                          // RT * (dv + 2): m, l, o
  float *osum = part + RT * (dv + 2);                                     // vrows * RT * dv
  __shared__ float m_run[RT], l_run[RT], corr[RT];
  pdl_prologue();

  const int tid = threadIdx.x, lane = tid % WARP, warp = tid / WARP;
  const int g = blockIdx.x / d.subs, sub = blockIdx.x % d.subs, b = blockIdx.y;
  const int sp = blockIdx.z, nsplit = gridDim.z;
  const int rep = a.H / a.G, r0 = sub * RT, nr = min(RT, rep - r0), h0 = g * rep + r0;
  const long long p = a.pos[b];
  const T *row = static_cast<const T *>(a.qkv) + (size_t)b * a.ld;
  const T *k_new = row + (size_t)(a.H + g) * dk;
  const T *v_new = row + (size_t)(a.H + a.G) * dk + (size_t)g * dv;
  T *kr = static_cast<T *>(d.k_ring) + ((size_t)b * a.G + g) * a.cap * dk;
  T *vr = static_cast<T *>(d.v_ring) + ((size_t)b * a.G + g) * a.cap * dv;

  long long lo = p - a.window + 1;
  if (lo < 0) lo = 0;
  const int len = (int)(p - lo + 1);
  const int chunk = (len + nsplit - 1) / nsplit;
  const int t_begin = min(len, sp * chunk), t_end = min(len, t_begin + chunk);
  const int slot0 = (int)(lo % a.cap);  // slot of the window's first token

  for (int i = tid; i < d.half; i += WD_THREADS) {
    float s, c;
    sincosf((float)p * d.freqs[i], &s, &c);
    cs[i] = c * d.amp;
    cs[d.half + i] = s * d.amp;
  }
  if (tid < RT) {
    m_run[tid] = -INFINITY;
    l_run[tid] = 0.f;
  }
  const int nkc = dk / N, nvc = dv / N;
  const int vch = tid % nvc, vrow = tid / nvc;  // value columns of this thread, and its first row
  float acc[RT][N];
#pragma unroll
  for (int r = 0; r < RT; ++r)
#pragma unroll
    for (int e = 0; e < N; ++e) acc[r][e] = 0.f;
  const bool wide_v = nvc > WD_THREADS;  // (element-wise form only: a thread then owns several columns, below)

  for (int p0 = t_begin; p0 < t_end; p0 += tile) {
    const int pn = min(tile, t_end - p0);
    for (int c = tid; c < pn * nkc; c += WD_THREADS) {
      const int t = c / nkc, j = c % nkc;
      if (p0 + t == len - 1) continue;  // the new token is not in the ring yet
      int slot = slot0 + p0 + t;
      if (slot >= a.cap) slot -= a.cap;
      if (VEC)
        cp_async16_zfill(smem_addr(k_sm + (size_t)t * d.k_pitch + j * N), kr + (size_t)slot * dk + j * N, 16);
      else
        k_sm[(size_t)t * d.k_pitch + j] = kr[(size_t)slot * dk + j];
    }
    for (int c = tid; c < pn * nvc; c += WD_THREADS) {
      const int t = c / nvc, j = c % nvc;
      if (p0 + t == len - 1) continue;
      int slot = slot0 + p0 + t;
      if (slot >= a.cap) slot -= a.cap;
      if (VEC)
        cp_async16_zfill(smem_addr(v_sm + (size_t)t * d.v_pitch + j * N), vr + (size_t)slot * dv + j * N, 16);
      else
        v_sm[(size_t)t * d.v_pitch + j] = vr[(size_t)slot * dv + j];
    }
    if (VEC) cp_async_commit();
    if (p0 == t_begin) __syncthreads();  // cs[] is complete
    if (p0 == t_begin)
      for (int i = tid; i < nr * dk; i += WD_THREADS)
        qs[i] = to_f(from_f<T>(rotated(row + (size_t)(h0 + i / dk) * dk, i % dk, cs, d.half)));
    if (p0 + pn == len) {  // this block holds the new token: the first head subgroup stores it
      const size_t slot = (size_t)(p % a.cap);
      for (int i = tid; i < dk; i += WD_THREADS) {
        const T k = from_f<T>(rotated(k_new, i, cs, d.half));
        k_sm[(size_t)(pn - 1) * d.k_pitch + i] = k;
        if (sub == 0) kr[slot * dk + i] = k;
      }
      for (int i = tid; i < dv; i += WD_THREADS) {
        v_sm[(size_t)(pn - 1) * d.v_pitch + i] = v_new[i];
        if (sub == 0) vr[slot * dv + i] = v_new[i];
      }
    }
    if (VEC) cp_async_wait<0>();
    __syncthreads();
    // scores: a thread per token
    for (int t = tid; t < tile; t += WD_THREADS) {
      float s[RT];
#pragma unroll
      for (int r = 0; r < RT; ++r) s[r] = 0.f;
      if (t < pn) {
        for (int c = 0; c < nkc; ++c) {
          float kf[N];
          if (VEC)
            unpack_chunk<T>(*reinterpret_cast<const uint4 *>(k_sm + (size_t)t * d.k_pitch + c * N), kf);
          else
            kf[0] = to_f(k_sm[(size_t)t * d.k_pitch + c]);
#pragma unroll
          for (int r = 0; r < RT; ++r)
#pragma unroll
            for (int e = 0; e < N; ++e) s[r] = fmaf(kf[e], r < nr ? qs[r * dk + c * N + e] : 0.f, s[r]);
        }
      }
#pragma unroll
      for (int r = 0; r < RT; ++r) sc[r * tile + t] = t < pn ? s[r] * a.scale : -INFINITY;
    }
    __syncthreads();
    for (int r = warp; r < nr; r += WD_THREADS / WARP) {
      float mx = m_run[r];
      for (int t = lane; t < pn; t += WARP) mx = fmaxf(mx, sc[r * tile + t]);
      mx = warp_max(mx);
      float sum = 0.f;
      for (int t = lane; t < pn; t += WARP) {
        const float w = expf(sc[r * tile + t] - mx);
        sc[r * tile + t] = w;
        sum += w;
      }
      sum = warp_sum(sum);
      if (lane == 0) {
        corr[r] = m_run[r] == -INFINITY ? 0.f : expf(m_run[r] - mx);
        l_run[r] = l_run[r] * corr[r] + sum;
        m_run[r] = mx;
      }
    }
    __syncthreads();
    if (!wide_v && vrow < d.vrows) {
#pragma unroll
      for (int r = 0; r < RT; ++r)
        if (r < nr) {
#pragma unroll
          for (int e = 0; e < N; ++e) acc[r][e] *= corr[r];
        }
      for (int t = vrow; t < pn; t += d.vrows) {
        float vf[N];
        if (VEC)
          unpack_chunk<T>(*reinterpret_cast<const uint4 *>(v_sm + (size_t)t * d.v_pitch + vch * N), vf);
        else
          vf[0] = to_f(v_sm[(size_t)t * d.v_pitch + vch]);
#pragma unroll
        for (int r = 0; r < RT; ++r) {
          if (r < nr) {
            const float w = sc[r * tile + t];
#pragma unroll
            for (int e = 0; e < N; ++e) acc[r][e] = fmaf(w, vf[e], acc[r][e]);
          }
        }
      }
    } else if (wide_v) {
      // more value columns than threads: sums live in shared memory (vrows == 1)
      for (int j = tid; j < nvc; j += WD_THREADS)
        for (int r = 0; r < nr; ++r) {
          float o = p0 == t_begin ? 0.f : osum[r * dv + j] * corr[r];
          for (int t = 0; t < pn; ++t) o = fmaf(sc[r * tile + t], to_f(v_sm[(size_t)t * d.v_pitch + j]), o);
          osum[r * dv + j] = o;
        }
    }
    __syncthreads();  // the tile and sc[] are reused
  }
  if (!wide_v && vrow < d.vrows) {
#pragma unroll
    for (int r = 0; r < RT; ++r)
#pragma unroll
      for (int e = 0; e < N; ++e) osum[((size_t)vrow * RT + r) * dv + vch * N + e] = acc[r][e];
  }
  __syncthreads();
  const bool empty = t_begin >= t_end;
  for (int i = tid; i < nr * dv; i += WD_THREADS) {
    const int r = i / dv, j = i % dv;
    float o = 0.f;
    if (!empty)
      for (int v = 0; v < d.vrows; ++v) o += osum[((size_t)v * RT + r) * dv + j];
    part[r * (dv + 2) + 2 + j] = o;
  }
  if (tid < nr) {
    part[tid * (dv + 2)] = m_run[tid];
    part[tid * (dv + 2) + 1] = l_run[tid];
  }
  cg::cluster_group cluster = cg::this_cluster();
  if (nsplit > 1)
    cluster.sync();
  else
    __syncthreads();
  if (sp == 0) {
    for (int i = tid; i < nr * dv; i += WD_THREADS) {
      const int r = i / dv, j = i % dv;
      const float sink = a.sink ? a.sink[h0 + r] : -INFINITY;
      float ms[WD_MAX_SPLITS], m = sink;
#pragma unroll
      for (int s = 0; s < WD_MAX_SPLITS; ++s) {
        ms[s] = -INFINITY;
        if (s < nsplit) ms[s] = *(nsplit > 1 ? cluster.map_shared_rank(part + r * (dv + 2), s) : part + r * (dv + 2));
        m = fmaxf(m, ms[s]);
      }
      float l = a.sink ? expf(sink - m) : 0.f, o = 0.f;
#pragma unroll
      for (int s = 0; s < WD_MAX_SPLITS; ++s) {
        if (s < nsplit && ms[s] != -INFINITY) {
          const float *q = (nsplit > 1 ? cluster.map_shared_rank(part, s) : part) + r * (dv + 2);
          const float w = expf(ms[s] - m);
          l = fmaf(w, q[1], l);
          o = fmaf(w, q[2 + j], o);
        }
      }
      static_cast<T *>(a.out)[((size_t)b * a.H + h0 + r) * dv + j] = from_f<T>(o / l);
    }
  }
  if (nsplit > 1) cluster.sync();  // no block leaves while rank 0 may still read its shared memory
}

template <typename T, int RT, bool VEC>
static int launch_decode(DecodeArgs d, int nsplit, cudaStream_t st) {
  const WindowArgs &a = d.w;
  constexpr int N = VEC ? Chunk<T>::N : 1;
  d.subs = ceil_div(a.H / a.G, RT);
  // an odd number of 16-byte units per row: rows of one column then fall into different banks
  auto pitch = [](int dim) {
    if (!VEC) return dim | 1;
    const int units = dim / N;
    return (units | 1) * N;
  };
  d.k_pitch = pitch(a.dk);
  d.v_pitch = pitch(a.dv);
  const int nvc = a.dv / N;
  d.vrows = nvc > WD_THREADS ? 1 : WD_THREADS / nvc;
  size_t smem = 0;
  for (d.tile = 128;; d.tile /= 2) {
    size_t kv = (size_t)d.tile * (d.k_pitch + d.v_pitch) * sizeof(T);
    kv = (kv + 15) / 16 * 16;
    smem = kv + 4 * ((size_t)RT * a.dk + (size_t)RT * d.tile + 2 * d.half + (size_t)RT * (a.dv + 2) +
                     (size_t)d.vrows * RT * a.dv);
    if (smem <= 200 * 1024) break;
    if (d.tile == 16) {
      set_error("window_attn_decode: head sizes %d / %d are too large", a.dk, a.dv);
      return DJV_ERR_UNSUPPORTED;
    }
  }
  if (!VEC && ((size_t)d.tile * (d.k_pitch + d.v_pitch) * sizeof(T)) % 4 != 0) return DJV_ERR_UNSUPPORTED;
  cudaFuncSetAttribute(window_decode_kernel<T, RT, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
  djv::launch_kernel_cluster(window_decode_kernel<T, RT, VEC>, dim3(a.G * d.subs, a.B, nsplit), dim3(WD_THREADS), smem,
                             st, dim3(1, 1, nsplit), d);
  count_launch();
  return check_launch("window_attn_decode");
}

template <typename T, bool VEC>
static int dispatch_decode(const DecodeArgs &d, int nsplit, cudaStream_t st) {
  const int rep = d.w.H / d.w.G;
  if (rep == 1) return launch_decode<T, 1, VEC>(d, nsplit, st);
  if (rep == 2) return launch_decode<T, 2, VEC>(d, nsplit, st);
  if (rep <= 4) return launch_decode<T, 4, VEC>(d, nsplit, st);
  return launch_decode<T, 8, VEC>(d, nsplit, st);
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

}  // namespace djv

using namespace djv;

static int check_window(const char *op, int dtype, const void *qkv, const void *k, const void *v, const long long *pos,
                        int B, int n, int H, int G, int dk, int dv, int cap, int window, long long ld) {
  DJV_REQUIRE(dtype == DJV_DTYPE_BF16 || dtype == DJV_DTYPE_F32, "%s: dtype %d", op, dtype);
  DJV_REQUIRE(qkv && k && v && pos, "%s: null pointer", op);
  DJV_REQUIRE(B >= 1 && B <= 65535 && n >= 1, "%s: B=%d n=%d", op, B, n);
  DJV_REQUIRE(G >= 1 && H >= G && H % G == 0 && H <= 65535, "%s: %d query heads over %d kv heads", op, H, G);
  DJV_REQUIRE(dk >= 1 && dv >= 1 && dk <= 512 && dv <= 512, "%s: head sizes %d / %d (up to 512)", op, dk, dv);
  DJV_REQUIRE(cap >= 1 && window >= 1, "%s: cap=%d window=%d", op, cap, window);
  DJV_REQUIRE(ld >= (long long)(H + G) * dk + (long long)G * dv, "%s: row stride %lld is too small", op, ld);
  return DJV_OK;
}

extern "C" int djv_rotary(int dtype, void *buf, long long ld, const float *freqs, float amp, const long long *pos, int B,
                          int n, int heads, int dim, int half, void *stream) {
  DJV_REQUIRE(dtype == DJV_DTYPE_BF16 || dtype == DJV_DTYPE_F32, "rotary: dtype %d", dtype);
  DJV_REQUIRE(buf && freqs && pos, "rotary: null pointer");
  DJV_REQUIRE(B >= 1 && n >= 1 && heads >= 1 && half >= 1 && 2 * half <= dim && half <= 4096 &&
                  ld >= (long long)heads * dim && (long long)B * n < (1ll << 31),
              "rotary: B=%d n=%d heads=%d dim=%d half=%d", B, n, heads, dim, half);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  int threads = ceil_div(heads * half, 4 * WARP) * WARP;
  threads = threads > 512 ? 512 : threads;
  if (dtype == DJV_DTYPE_BF16)
    djv::launch_kernel(rotary_kernel<bf16>, B * n, threads, half * 8, st, static_cast<bf16 *>(buf), ld, freqs, amp, pos,
                       n, heads, dim, half);
  else
    djv::launch_kernel(rotary_kernel<float>, B * n, threads, half * 8, st, static_cast<float *>(buf), ld, freqs, amp,
                       pos, n, heads, dim, half);
  count_launch();
  return check_launch("rotary");
}

extern "C" int djv_window_attn(int dtype, void *out, const void *qkv, long long ld, const void *k_ring,
                               const void *v_ring, const float *sink, const long long *pos, int B, int n, int H, int G,
                               int dk, int dv, int cap, int window, float scale, void *stream) {
  int rc = check_window("window_attn", dtype, qkv, k_ring, v_ring, pos, B, n, H, G, dk, dv, cap, window, ld);
  if (rc) return rc;
  DJV_REQUIRE(out, "window_attn: null output");
  if (window > cap) window = cap;  // a ring that is shorter than the window holds the longest sequence
  const WindowArgs a{out, qkv, ld, k_ring, v_ring, sink, pos, B, n, H, G, dk, dv, cap, window, scale};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (dtype == DJV_DTYPE_BF16) return window_prefill_supported(a) ? window_prefill(a, st) : launch_simple<bf16>(a, st);
  return launch_simple<float>(a, st);
}

extern "C" int djv_window_store(int dtype, void *k_ring, void *v_ring, const void *qkv, long long ld,
                                const long long *pos, int B, int n, int H, int G, int dk, int dv, int cap,
                                void *stream) {
  int rc = check_window("window_store", dtype, qkv, k_ring, v_ring, pos, B, n, H, G, dk, dv, cap, 1, ld);
  if (rc) return rc;
  const int cnt = n < cap ? n : cap;
  const dim3 grid(cnt, B);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (dtype == DJV_DTYPE_BF16)
    djv::launch_kernel(window_store_kernel<bf16>, grid, dim3(128), 0, st, static_cast<bf16 *>(k_ring),
                       static_cast<bf16 *>(v_ring), static_cast<const bf16 *>(qkv), ld, pos, n, H, G, dk, dv, cap,
                       n - cnt);
  else
    djv::launch_kernel(window_store_kernel<float>, grid, dim3(128), 0, st, static_cast<float *>(k_ring),
                       static_cast<float *>(v_ring), static_cast<const float *>(qkv), ld, pos, n, H, G, dk, dv, cap,
                       n - cnt);
  count_launch();
  return check_launch("window_store");
}

extern "C" int djv_window_attn_decode(int dtype, void *out, const void *qkv, long long ld, void *k_ring, void *v_ring,
                                      const float *sink, const float *freqs, float amp, int half, const long long *pos,
                                      int B, int H, int G, int dk, int dv, int cap, int window, float scale,
                                      void *stream) {
  int rc = check_window("window_attn_decode", dtype, qkv, k_ring, v_ring, pos, B, 1, H, G, dk, dv, cap, window, ld);
  if (rc) return rc;
  DJV_REQUIRE(out, "window_attn_decode: null output");
  if (!freqs) half = 0;
  DJV_REQUIRE(half >= 0 && 2 * half <= dk, "window_attn_decode: %d rotary pairs in %d dimensions", half, dk);
  if (window > cap) window = cap;
  DecodeArgs d = {};
  d.w = WindowArgs{out, qkv, ld, k_ring, v_ring, sink, pos, B, 1, H, G, dk, dv, cap, window, scale};
  d.k_ring = k_ring;
  d.v_ring = v_ring;
  d.freqs = freqs;
  d.amp = amp;
  d.half = half;
  int nsplit = 1;
  while (nsplit < WD_MAX_SPLITS && window > 64 * nsplit) nsplit *= 2;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (dtype == DJV_DTYPE_BF16) {
    const bool vec = dk % 8 == 0 && dv % 8 == 0 && dv / 8 <= WD_THREADS && aligned16(k_ring) && aligned16(v_ring);
    return vec ? dispatch_decode<bf16, true>(d, nsplit, st) : dispatch_decode<bf16, false>(d, nsplit, st);
  }
  const bool vec = dk % 4 == 0 && dv % 4 == 0 && dv / 4 <= WD_THREADS && aligned16(k_ring) && aligned16(v_ring);
  return vec ? dispatch_decode<float, true>(d, nsplit, st) : dispatch_decode<float, false>(d, nsplit, st);
}
