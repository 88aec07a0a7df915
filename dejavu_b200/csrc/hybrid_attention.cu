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
#include <math.h>

#include "../../include/dejavu_b200_hybrid.h"
#include "hybrid_attention.cuh"
#include "dtype.cuh"

namespace djv {

namespace cg = cooperative_groups;

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
// grid (G * head subgroups, B, splits); the splits of the window form a cluster and push their partial sums into rank
// 0's shared memory, which combines them. A block takes RT query heads of one kv head, so K and V are read once for all
// of them. A pass covers TILE tokens: all its K and V loads are issued before anything waits on them.
constexpr int WD_THREADS = 256;
constexpr int WD_MAX_SPLITS = 8;

struct DecodeArgs {
  WindowArgs w;
  void *k_ring, *v_ring;
  const float *freqs;
  float amp;
  int half, subs;
};

// rotated element i of a head vector
__device__ __forceinline__ float rotated(const float *x, int i, const float *cs, int half) {
  const float u = x[i];
  if (i < half) return u * cs[i] - x[i + half] * cs[half + i];
  if (i < 2 * half) return u * cs[i - half] + x[i - half] * cs[i];
  return u;
}

// KL: 16-byte chunks of a key per lane (8 lanes per key); VI: 16-byte chunks of values per thread and pass.
// KL == 0: any head size and alignment, element by element, one token of K and one column of V per thread at a time.
template <typename T, int RT, int KL, int VI>
__global__ void __launch_bounds__(WD_THREADS) window_decode_kernel(DecodeArgs d) {
  const WindowArgs &a = d.w;
  constexpr bool VEC = KL > 0;
  constexpr int N = VEC ? Chunk<T>::N : 1;
  constexpr int TILE = sizeof(T) == 2 ? 128 : 64;
  constexpr int KT = TILE / (WD_THREADS / 8);  // keys per group of 8 lanes and pass
  extern __shared__ __align__(16) float sm[];
  const int dk = a.dk, dv = a.dv, ps = RT * (dv + 2);
  float *qs = sm;                        // RT * dk
  float *sc = qs + RT * ((dk + 3) & ~3); // RT * TILE
  T *kn = reinterpret_cast<T *>(sc + RT * TILE);                        // the new token's rotated key
  float *cs = reinterpret_cast<float *>(kn) + ((dk + 3) & ~3);          // 2 * half
  float *raw = cs + 2 * ((d.half + 1) & ~1);                            // the heads' queries and the key, not rotated
  float *part = raw + (RT + 1) * dk;                                    // splits * RT * (m, l, o[dv])
  const int nvc = VEC ? dv / N : min(dv, WD_THREADS);
  const int vrows = WD_THREADS / nvc;
  float *osum = part + WD_MAX_SPLITS * ps;  // vrows * RT * dv
  __shared__ float m_run[RT], l_run[RT], corr[RT];
  cg::cluster_group cluster = cg::this_cluster();
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  const int nsplit = gridDim.z;
  if (nsplit > 1) cluster.barrier_arrive();  // (waited for before the first access to another block's memory)
  asm volatile("griddepcontrol.wait;" ::: "memory");

  const int tid = threadIdx.x, lane = tid % WARP, warp = tid / WARP;
  const int g = blockIdx.x / d.subs, sub = blockIdx.x % d.subs, b = blockIdx.y, sp = blockIdx.z;
  const int rep = a.H / a.G, r0 = sub * RT, nr = min(RT, rep - r0), h0 = g * rep + r0;
  const long long p = a.pos[b];
  const T *row = static_cast<const T *>(a.q) + (size_t)b * a.ldq;
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
  auto slot_of = [&](int t) {
    const int s = slot0 + t;
    return (size_t)(s >= a.cap ? s - a.cap : s);
  };

  const int ksub = tid % 8, kgrp = tid / 8;
  const int vch = tid % nvc, vrow = tid / nvc;
  const bool vmine = vrow < vrows;
  const int nkc = dk / N;
  uint4 kreg[KT][VEC ? KL : 1], vreg[VEC ? VI : 1];
  const uint4 zero = make_uint4(0, 0, 0, 0);
  auto fetch = [&](int p0) {
    if (VEC) {
#pragma unroll
      for (int x = 0; x < KT; ++x) {
        const int t = p0 + x * (WD_THREADS / 8) + kgrp;
        const uint4 *src = reinterpret_cast<const uint4 *>(kr + slot_of(t) * dk);
#pragma unroll
        for (int c = 0; c < KL; ++c)  // the last token of the window is not in the ring yet
          kreg[x][c] = (t < t_end && t < len - 1 && ksub + c * 8 < nkc) ? src[ksub + c * 8] : zero;
      }
#pragma unroll
      for (int x = 0; x < VI; ++x) {
        const int i = x * vrows + vrow, t = p0 + i;
        vreg[x] = zero;
        if (vmine && i < TILE && t < t_end)
          vreg[x] = t < len - 1 ? *reinterpret_cast<const uint4 *>(vr + slot_of(t) * dv + vch * N)
                                : *reinterpret_cast<const uint4 *>(v_new + vch * N);
      }
    }
  };
  fetch(t_begin);
  for (int i = tid; i < nr * dk; i += WD_THREADS) raw[i] = to_f(row[(size_t)h0 * dk + i]);
  for (int i = tid; i < dk; i += WD_THREADS) raw[RT * dk + i] = to_f(k_new[i]);

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
  __syncthreads();
  for (int i = tid; i < RT * dk; i += WD_THREADS) {
    const int r = i / dk;
    qs[i] = r < nr ? to_f(from_f<T>(rotated(raw + r * dk, i - r * dk, cs, d.half))) : 0.f;
  }
  if (t_end == len && t_begin < t_end) {  // this block holds the new token: the first head subgroup stores it
    const size_t slot = (size_t)(p % a.cap);
    for (int i = tid; i < dk; i += WD_THREADS) {
      const T k = from_f<T>(rotated(raw + RT * dk, i, cs, d.half));
      kn[i] = k;
      if (sub == 0) kr[slot * dk + i] = k;
    }
    if (sub == 0)
      for (int i = tid; i < dv; i += WD_THREADS) vr[slot * dv + i] = v_new[i];
  }
  __syncthreads();

  float acc[RT][N];
#pragma unroll
  for (int r = 0; r < RT; ++r)
#pragma unroll
    for (int e = 0; e < N; ++e) acc[r][e] = 0.f;

  for (int p0 = t_begin; p0 < t_end; p0 += TILE) {
    const int pn = min(TILE, t_end - p0);
    if (VEC) {
      if (p0 != t_begin) fetch(p0);
      float s[KT][RT];
#pragma unroll
      for (int x = 0; x < KT; ++x)
#pragma unroll
        for (int r = 0; r < RT; ++r) s[x][r] = 0.f;
#pragma unroll
      for (int c = 0; c < (VEC ? KL : 1); ++c) {
        const int ch = ksub + c * 8;
        if (ch >= nkc) continue;
        float kf[KT][N];
#pragma unroll
        for (int x = 0; x < KT; ++x) {
          if (p0 + x * (WD_THREADS / 8) + kgrp == len - 1) kreg[x][c] = *reinterpret_cast<const uint4 *>(kn + ch * N);
          if constexpr (VEC) unpack_chunk<T>(kreg[x][c], kf[x]);
        }
#pragma unroll
        for (int r = 0; r < RT; ++r) {
          float qf[N];
#pragma unroll
          for (int e = 0; e < N; ++e) qf[e] = qs[r * dk + ch * N + e];
#pragma unroll
          for (int x = 0; x < KT; ++x)
#pragma unroll
            for (int e = 0; e < N; ++e) s[x][r] = fmaf(kf[x][e], qf[e], s[x][r]);
        }
      }
#pragma unroll
      for (int x = 0; x < KT; ++x) {
        const int t = x * (WD_THREADS / 8) + kgrp;
#pragma unroll
        for (int r = 0; r < RT; ++r) {
          float v = s[x][r];
          v += __shfl_xor_sync(0xffffffffu, v, 4);
          v += __shfl_xor_sync(0xffffffffu, v, 2);
          v += __shfl_xor_sync(0xffffffffu, v, 1);
          if (ksub == 0) sc[r * TILE + t] = t < pn ? v * a.scale : -INFINITY;
        }
      }
    } else {
      for (int i = tid; i < RT * TILE; i += WD_THREADS) {
        const int r = i / TILE, t = i % TILE;
        float v = -INFINITY;
        if (t < pn && r < nr) {
          const T *k = p0 + t == len - 1 ? kn : kr + slot_of(p0 + t) * dk;
          v = 0.f;
          for (int c = 0; c < dk; ++c) v = fmaf(to_f(k[c]), qs[r * dk + c], v);
          v *= a.scale;
        }
        sc[i] = v;
      }
    }
    __syncthreads();
    for (int r = warp; r < nr; r += WD_THREADS / WARP) {
      float x[TILE / WARP], mx = m_run[r];
#pragma unroll
      for (int i = 0; i < TILE / WARP; ++i) {
        x[i] = sc[r * TILE + i * WARP + lane];
        mx = fmaxf(mx, x[i]);
      }
      mx = warp_max(mx);
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < TILE / WARP; ++i) {
        const float w = expf(x[i] - mx);  // 0 past the end of the pass
        sc[r * TILE + i * WARP + lane] = w;
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
    if (VEC) {
      if (p0 != t_begin) {
#pragma unroll
        for (int r = 0; r < RT; ++r) {
          const float w = r < nr ? corr[r] : 0.f;
#pragma unroll
          for (int e = 0; e < N; ++e) acc[r][e] *= w;
        }
      }
#pragma unroll
      for (int x = 0; x < (VEC ? VI : 1); ++x) {
        const int i = x * vrows + vrow;
        float vf[N];
        if constexpr (VEC) unpack_chunk<T>(vreg[x], vf);
        if (vmine && i < pn) {
#pragma unroll
          for (int r = 0; r < RT; ++r) {
            const float w = r < nr ? sc[r * TILE + i] : 0.f;
#pragma unroll
            for (int e = 0; e < N; ++e) acc[r][e] = fmaf(w, vf[e], acc[r][e]);
          }
        }
      }
    } else {
      for (int j = tid; j < dv; j += WD_THREADS)  // sums in shared memory, one thread per column
        for (int r = 0; r < nr; ++r) {
          float o = p0 == t_begin ? 0.f : osum[r * dv + j] * corr[r];
          for (int t = 0; t < pn; ++t) {
            const T *v = p0 + t == len - 1 ? v_new : vr + slot_of(p0 + t) * dv;
            o = fmaf(sc[r * TILE + t], to_f(v[j]), o);
          }
          osum[r * dv + j] = o;
        }
    }
    __syncthreads();  // sc[] is reused
  }
  const bool empty = t_begin >= t_end;
  if (VEC && vmine) {
#pragma unroll
    for (int r = 0; r < RT; ++r)
#pragma unroll
      for (int e = 0; e < N; ++e) osum[((size_t)vrow * RT + r) * dv + vch * N + e] = acc[r][e];
  }
  __syncthreads();
  if (nsplit > 1) cluster.barrier_wait();
  float *dst = (nsplit > 1 ? cluster.map_shared_rank(part, 0) : part) + sp * ps;
  for (int i = tid; i < nr * dv; i += WD_THREADS) {
    const int r = i / dv, j = i - r * dv;
    float o = 0.f;
    if (!empty)
      for (int v = 0; v < (VEC ? vrows : 1); ++v) o += osum[((size_t)v * RT + r) * dv + j];
    dst[r * (dv + 2) + 2 + j] = o;
  }
  if (tid < nr) {
    dst[tid * (dv + 2)] = m_run[tid];
    dst[tid * (dv + 2) + 1] = l_run[tid];
  }
  if (nsplit > 1)
    cluster.sync();
  else
    __syncthreads();
  if (sp != 0) return;
  for (int i = tid; i < nr * dv; i += WD_THREADS) {
    const int r = i / dv, j = i - r * dv;
    const float sink = a.sink ? a.sink[h0 + r] : -INFINITY;
    float ms[WD_MAX_SPLITS], m = sink;
#pragma unroll
    for (int s = 0; s < WD_MAX_SPLITS; ++s) {
      ms[s] = s < nsplit ? part[s * ps + r * (dv + 2)] : -INFINITY;
      m = fmaxf(m, ms[s]);
    }
    float l = a.sink ? expf(sink - m) : 0.f, o = 0.f;
#pragma unroll
    for (int s = 0; s < WD_MAX_SPLITS; ++s) {
      if (s < nsplit && ms[s] != -INFINITY) {
        const float *q = part + s * ps + r * (dv + 2);
        const float w = expf(ms[s] - m);
        l = fmaf(w, q[1], l);
        o = fmaf(w, q[2 + j], o);
      }
    }
    static_cast<T *>(a.out)[((size_t)b * a.H + h0 + r) * dv + j] = from_f<T>(o / l);
  }
}

template <typename T, int RT, int KL, int VI>
static int launch_decode(DecodeArgs d, int nsplit, cudaStream_t st) {
  const WindowArgs &a = d.w;
  constexpr int TILE = sizeof(T) == 2 ? 128 : 64;
  d.subs = ceil_div(a.H / a.G, RT);
  const int nvc = KL > 0 ? a.dv / Chunk<T>::N : WD_THREADS;
  const size_t dk4 = (a.dk + 3) & ~3;
  const size_t smem = 4 * (RT * dk4 + (size_t)RT * TILE + dk4 + 2 * ((d.half + 1) & ~1) + (size_t)(RT + 1) * a.dk +
                           (size_t)WD_MAX_SPLITS * RT * (a.dv + 2) + (size_t)(WD_THREADS / nvc) * RT * a.dv);
  if (smem > 220 * 1024) {
    set_error("window_attn_decode: head sizes %d / %d are too large", a.dk, a.dv);
    return DJV_ERR_UNSUPPORTED;
  }
  cudaFuncSetAttribute(window_decode_kernel<T, RT, KL, VI>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
  djv::launch_kernel_cluster(window_decode_kernel<T, RT, KL, VI>, dim3(a.G * d.subs, a.B, nsplit), dim3(WD_THREADS), smem,
                             st, dim3(1, 1, nsplit), d);
  count_launch();
  return check_launch("window_attn_decode");
}

template <typename T, int RT>
static int dispatch_decode(const DecodeArgs &d, int nsplit, bool vec, cudaStream_t st) {
  if (!vec) return launch_decode<T, RT, 0, 0>(d, nsplit, st);
  constexpr int N = Chunk<T>::N, TILE = sizeof(T) == 2 ? 128 : 64;
  const int kl = ceil_div(d.w.dk / N, 8);
  const int vi = ceil_div(TILE, WD_THREADS / (d.w.dv / N));
  // (the larger instance of each pair serves the sizes between)
  if (kl <= 2 && vi <= 8) return launch_decode<T, RT, 2, 8>(d, nsplit, st);
  if (kl <= 4 && vi <= 16) return launch_decode<T, RT, 4, 16>(d, nsplit, st);
  if (sizeof(T) == 4 && kl <= 8 && vi <= 16) return launch_decode<T, RT, sizeof(T) == 4 ? 8 : 4, 16>(d, nsplit, st);
  return launch_decode<T, RT, 0, 0>(d, nsplit, st);
}

template <typename T>
static int dispatch_decode(const DecodeArgs &d, int max_split, bool vec, cudaStream_t st) {
  // Query heads per block (rt) and splits of the window: waves of blocks times passes of a block times a pass's work,
  // which is a part for the K and V loads and one per query head. Blocks of one or two heads fit a multiprocessor
  // twice; clusters of 8 leave some multiprocessors unused (120 of 148 hold one).
  const int rep = d.w.H / d.w.G, tile = sizeof(T) == 2 ? 128 : 64;
  int rt = 8, nsplit = max_split;
  double best = 1e30;
  for (int ns = max_split; ns >= 1; ns /= 2) {
    for (int r = 1; r <= 8 && (r == 1 || r / 2 < rep); r *= 2) {
      const double room = (r <= 2 ? 2.0 : 1.0) * sm_count() * (ns == 8 ? 0.81 : (ns > 1 ? 0.89 : 1.0));
      const double waves = ceil((double)d.w.G * ceil_div(rep, r) * d.w.B * ns / room);
      const double cost = waves * ceil_div(ceil_div(d.w.window, ns), tile) * (2 + r);
      if (cost < best) {
        best = cost;
        rt = r;
        nsplit = ns;
      }
    }
  }
  if (rt == 1) return dispatch_decode<T, 1>(d, nsplit, vec, st);
  if (rt == 2) return dispatch_decode<T, 2>(d, nsplit, vec, st);
  if (rt == 4) return dispatch_decode<T, 4>(d, nsplit, vec, st);
  return dispatch_decode<T, 8>(d, nsplit, vec, st);
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

// q, k and v side by side in the rows of one projection, earlier tokens in the rings
static WindowArgs fused_args(int dtype, void *out, const void *qkv, long long ld, const void *k_ring, const void *v_ring,
                             const float *sink, const long long *pos, int B, int n, int H, int G, int dk, int dv, int cap,
                             int window, float scale) {
  const char *k = static_cast<const char *>(qkv) + (size_t)H * dk * dtype_bytes(dtype);
  const char *v = k + (size_t)G * dk * dtype_bytes(dtype);
  return WindowArgs{out, qkv, ld, k, ld, v, ld, nullptr, 0, 0, nullptr, 0, k_ring, v_ring, sink, pos, B, n, H, G, dk, dv,
                    cap, 0, window, scale};
}

extern "C" int djv_window_attn(int dtype, void *out, const void *qkv, long long ld, const void *k_ring,
                               const void *v_ring, const float *sink, const long long *pos, int B, int n, int H, int G,
                               int dk, int dv, int cap, int window, float scale, void *stream) {
  int rc = check_window("window_attn", dtype, qkv, k_ring, v_ring, pos, B, n, H, G, dk, dv, cap, window, ld);
  if (rc) return rc;
  DJV_REQUIRE(out, "window_attn: null output");
  if (window > cap) window = cap;  // a ring that is shorter than the window holds the longest sequence
  const WindowArgs a = fused_args(dtype, out, qkv, ld, k_ring, v_ring, sink, pos, B, n, H, G, dk, dv, cap, window, scale);
  return window_attn_portion(dtype, a, static_cast<cudaStream_t>(stream));
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
  d.w = fused_args(dtype, out, qkv, ld, k_ring, v_ring, sink, pos, B, 1, H, G, dk, dv, cap, window, scale);
  d.k_ring = k_ring;
  d.v_ring = v_ring;
  d.freqs = freqs;
  d.amp = amp;
  d.half = half;
  int nsplit = 1;
  while (nsplit < WD_MAX_SPLITS && window > 64 * nsplit) nsplit *= 2;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int chunk = 16 / (int)dtype_bytes(dtype);
  const bool vec = dk % chunk == 0 && dv % chunk == 0 && dv / chunk <= WD_THREADS && ld % chunk == 0 &&
                   aligned16(qkv) && aligned16(k_ring) && aligned16(v_ring);
  if (dtype == DJV_DTYPE_BF16) return dispatch_decode<bf16>(d, nsplit, vec, st);
  return dispatch_decode<float>(d, nsplit, vec, st);
}
