// Matrix memory (mLSTM): per head a (dk, dv) fp32 state S, a normaliser n (dk) and a running maximum m, with scalar gates
// given by their logarithms i_t and f_t:
//   m_t = max(f_t + m_(t-1), i_t),  S_t = e^(f_t + m_(t-1) - m_t) S_(t-1) + e^(i_t - m_t) k_t v_t^T,  n_t the same with k_t,
//   o_t = S_t^T q_t / (max(|n_t . q_t|, e^(-m_t)) + 1e-6),
// followed by an RMS norm over dv and a sigmoid gate.
//
// A portion of tokens is cut into chunks of C. With F_t the sum of f over the chunk up to and including t, a_s = i_s - F_s
// and M_t = max(m_in, a_0 .. a_t), the recurrence is m_t = F_t + M_t and
//   S_t = e^(m_in - M_t) S_in + sum_(s <= t) e^(a_s - M_t) k_s v_s^T      (n_t likewise),
// with no exponent above 0. Three kernels: every chunk's own contribution relative to its largest a (chunks in parallel),
// a scan over the chunks that turns contributions into incoming states, every chunk's outputs (in parallel, norm and gate
// included). The kernels here do the chunks' products in fp32 on the CUDA cores, for any head size and both element
// types; the tensor-core form for bf16 is in hybrid_mlstm_prefill.cu.
#include <cooperative_groups.h>

#include "../../include/dejavu_b200_routed.h"
#include "hybrid_mlstm.cuh"

namespace djv {

namespace cg = cooperative_groups;

constexpr float ML_DEN_EPS = 1e-6f;

// sizes rounded up to whole 4x4 register tiles
__host__ __device__ __forceinline__ int up4(int v) { return (v + 3) & ~3; }

template <typename T>
__global__ void __launch_bounds__(ML_THREADS) mlstm_chunk_state_kernel(MlstmArgs a) {
  extern __shared__ float sm[];
  __shared__ float2 as[64];
  __shared__ float2 amax;
  pdl_prologue();
  const int tid = threadIdx.x;
  const int ci = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
  const int dk = a.dk, dv = a.dv, dkp = up4(dk), dvp = up4(dv);
  const int t0 = ci * a.C, cl = min(a.C, a.n - t0);
  float *ks = sm, *vs = ks + a.C * dkp;  // [C][dkp], [C][dvp]
  const T *rows = static_cast<const T *>(a.proj) + ((size_t)b * a.n + t0) * a.ld;
  const int koff = a.H * dk + h * dk, voff = 2 * a.H * dk + h * dv;
  const size_t at = ((size_t)b * a.H + h) * a.nc + ci;
  if (tid < WARP) {
    double total, top;
    chunk_gates<2>(a, b, h, t0, cl, as, nullptr, nullptr, total, top);
    if (tid == 0) {
      amax = split_double(top);
      a.chunk[at * 3] = total;
      a.chunk[at * 3 + 1] = top;
    }
  }
  for (int i = tid; i < cl * dvp; i += ML_THREADS) {
    const int t = i / dvp, j = i % dvp;
    vs[i] = j < dv ? to_f(rows[(size_t)t * a.ld + voff + j]) : 0.f;
  }
  __syncthreads();
  for (int i = tid; i < cl * dkp; i += ML_THREADS) {
    const int t = i / dkp, c = i % dkp;
    ks[i] = c < dk ? to_f(rows[(size_t)t * a.ld + koff + c]) * exp_diff(as[t], amax) : 0.f;
  }
  __syncthreads();
  float *U = a.contrib + at * mlstm_contrib_stride(dk, dv);
  const int tk = dkp / 4, tv = dvp / 4;
  for (int tile = tid; tile < tk * tv; tile += ML_THREADS) {
    const int c0 = tile / tv * 4, j0 = tile % tv * 4;
    float acc[4][4] = {};
    for (int t = 0; t < cl; ++t) {
      const float4 k4 = *reinterpret_cast<const float4 *>(ks + t * dkp + c0);
      const float4 v4 = *reinterpret_cast<const float4 *>(vs + t * dvp + j0);
      const float kk[4] = {k4.x, k4.y, k4.z, k4.w}, vv[4] = {v4.x, v4.y, v4.z, v4.w};
#pragma unroll
      for (int x = 0; x < 4; ++x)
#pragma unroll
        for (int y = 0; y < 4; ++y) acc[x][y] = fmaf(kk[x], vv[y], acc[x][y]);
    }
#pragma unroll
    for (int x = 0; x < 4; ++x)
#pragma unroll
      for (int y = 0; y < 4; ++y)
        if (c0 + x < dk && j0 + y < dv) U[(size_t)(c0 + x) * dv + j0 + y] = acc[x][y];
  }
  for (int c = tid; c < dk; c += ML_THREADS) {
    float s = 0.f;
    for (int t = 0; t < cl; ++t) s += ks[t * dkp + c];
    U[(size_t)dk * dv + c] = s;
  }
}

// Contributions -> incoming states, V neighbouring elements per thread, chunks in order. SPLIT: the incoming S goes out
// as two bf16 terms (n stays where it is, in fp32).
template <int V, bool SPLIT>
__global__ void __launch_bounds__(ML_THREADS) mlstm_scan_kernel(MlstmArgs a) {
  pdl_prologue();
  const int per = a.dk * a.dv, all = per + a.dk;
  const int e = (blockIdx.x * ML_THREADS + threadIdx.x) * V;
  const int h = blockIdx.y, b = blockIdx.z;
  if (e >= all) return;
  const size_t bh = (size_t)b * a.H + h, cs = mlstm_contrib_stride(a.dk, a.dv);
  float *st = a.state + bh * mlstm_state_stride(a.dk, a.dv);
  double *ch = a.chunk + bh * a.nc * 3;
  auto get = [](const float *p, float (&v)[V]) {
    if (V == 4) {
      const float4 t = *reinterpret_cast<const float4 *>(p);
      v[0] = t.x; v[1 % V] = t.y; v[2 % V] = t.z; v[3 % V] = t.w;
    } else {
      v[0] = *p;
    }
  };
  auto put = [](float *p, const float (&v)[V]) {
    if (V == 4)
      *reinterpret_cast<float4 *>(p) = make_float4(v[0], v[1 % V], v[2 % V], v[3 % V]);
    else
      *p = v[0];
  };
  const bool fresh = a.pos[b] == 0;
  double m = fresh ? 0.0 : (double)st[all];
  float s[V];
#pragma unroll
  for (int v = 0; v < V; ++v) s[v] = 0.f;
  if (!fresh) get(st + e, s);
  float *U = a.contrib + bh * a.nc * cs + e;
  constexpr int CH = V == 4 ? 4 : 8;  // chunks whose loads are in flight together
  for (int c0 = 0; c0 < a.nc; c0 += CH) {
    float u[CH][V];
    double f[CH], top[CH];
#pragma unroll
    for (int c = 0; c < CH; ++c) {
      if (c0 + c < a.nc) {
        get(U + (size_t)(c0 + c) * cs, u[c]);
        f[c] = ch[(c0 + c) * 3];
        top[c] = ch[(c0 + c) * 3 + 1];
      }
    }
#pragma unroll
    for (int c = 0; c < CH; ++c) {
      if (c0 + c < a.nc) {
        if (SPLIT && e < per) {
          bf16 *hi = a.s_hi + (bh * a.nc + c0 + c) * per + e, *lo = a.s_lo + (bh * a.nc + c0 + c) * per + e;
          if (V == 4) {
            uint2 x, y;
            x.x = pack_bf16(s[0], s[1 % V]);
            x.y = pack_bf16(s[2 % V], s[3 % V]);
            const float2 r0 = b2f(x.x), r1 = b2f(x.y);
            y.x = pack_bf16(s[0] - r0.x, s[1 % V] - r0.y);
            y.y = pack_bf16(s[2 % V] - r1.x, s[3 % V] - r1.y);
            *reinterpret_cast<uint2 *>(hi) = x;
            *reinterpret_cast<uint2 *>(lo) = y;
          } else {
            const bf16 x = from_f<bf16>(s[0]);
            *hi = x;
            *lo = from_f<bf16>(s[0] - to_f(x));
          }
        } else {
          put(U + (size_t)(c0 + c) * cs, s);
        }
        if (e == 0) ch[(c0 + c) * 3 + 2] = m;
        const double M = fmax(m, top[c]);
        const float keep = expf((float)(m - M)), add = expf((float)(top[c] - M));
        m = f[c] + M;
#pragma unroll
        for (int v = 0; v < V; ++v) s[v] = fmaf(keep, s[v], add * u[c][v]);
      }
    }
  }
  put(st + e, s);
}

// the running maximum after the portion: by itself, because every thread of the scan reads the old one
__global__ void mlstm_finish_kernel(MlstmArgs a) {
  pdl_prologue();
  const int i = blockIdx.x * blockDim.x + threadIdx.x;  // (sequence, head)
  if (i >= a.B * a.H) return;
  const double *last = a.chunk + ((size_t)i * a.nc + a.nc - 1) * 3;
  a.state[(size_t)i * mlstm_state_stride(a.dk, a.dv) + (size_t)a.dk * a.dv + a.dk] = (float)(last[0] + fmax(last[2], last[1]));
}

template <typename T>
__global__ void __launch_bounds__(ML_THREADS) mlstm_chunk_out_kernel(MlstmArgs a) {
  extern __shared__ float sm[];
  __shared__ float2 as[64], mt[64];
  __shared__ double run[64], fs[64];
  __shared__ float w_in[64], floor_s[64], den[64];
  pdl_prologue();
  const int tid = threadIdx.x, lane = tid % WARP, warp = tid / WARP;
  const int ci = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
  const int dk = a.dk, dv = a.dv, C = a.C, dvp = up4(dv), kp = dk | 1;
  const int t0 = ci * C, cl = min(C, a.n - t0);
  float *qs = sm, *ks = qs + C * kp, *A = ks + C * kp;  // [C][kp] x2, [C][C]
  float *vs = sm + up4((int)(A + C * C - sm));          // [C][dvp]
  float *os = vs + C * dvp;                             // [C][dvp]
  const T *rows = static_cast<const T *>(a.proj) + ((size_t)b * a.n + t0) * a.ld;
  const int qoff = h * dk, koff = a.H * dk + h * dk, voff = 2 * a.H * dk + h * dv, goff = voff + a.H * dv;
  const size_t at = ((size_t)b * a.H + h) * a.nc + ci;
  if (warp == 0) {
    double total, top;
    chunk_gates<2>(a, b, h, t0, cl, as, run, fs, total, top);
    __syncwarp();
    const double m_in = a.chunk[at * 3 + 2];
    for (int t = lane; t < C; t += WARP) {
      const double M = fmax(run[t], m_in);
      mt[t] = split_double(M);
      w_in[t] = expf((float)(m_in - M));
      floor_s[t] = expf((float)-(fs[t] + M));
    }
  }
  for (int i = tid; i < cl * dk; i += ML_THREADS) {
    const int t = i / dk, c = i % dk;
    const T *r = rows + (size_t)t * a.ld;
    qs[t * kp + c] = to_f(r[qoff + c]) * a.scale;
    ks[t * kp + c] = to_f(r[koff + c]);
  }
  for (int i = tid; i < cl * dvp; i += ML_THREADS) {
    const int t = i / dvp, j = i % dvp;
    vs[i] = j < dv ? to_f(rows[(size_t)t * a.ld + voff + j]) : 0.f;
  }
  __syncthreads();
  for (int i = tid; i < cl * cl; i += ML_THREADS) {
    const int t = i / cl, s = i % cl;
    float acc = 0.f;
    if (s <= t) {
      for (int c = 0; c < dk; ++c) acc = fmaf(qs[t * kp + c], ks[s * kp + c], acc);
      acc *= exp_diff(as[s], mt[t]);
    }
    A[t * C + s] = acc;
  }
  __syncthreads();
  const float *S = a.contrib + at * mlstm_contrib_stride(dk, dv), *N = S + (size_t)dk * dv;
  for (int i = tid; i < cl * dk; i += ML_THREADS) {
    const int t = i / dk, c = i % dk;
    qs[t * kp + c] *= w_in[t];
  }
  __syncthreads();
  for (int t = warp; t < cl; t += ML_THREADS / WARP) {
    float s = 0.f;
    for (int c = lane; c < dk; c += WARP) s = fmaf(qs[t * kp + c], N[c], s);
    for (int c = lane; c <= t; c += WARP) s += A[t * C + c];
    s = warp_sum(s);
    if (lane == 0) den[t] = fmaxf(fabsf(s), floor_s[t]) + ML_DEN_EPS;
  }
  const int tt = (cl + 3) / 4, tv = dvp / 4;
  for (int tile = tid; tile < tt * tv; tile += ML_THREADS) {
    const int r0 = tile / tv * 4, j0 = tile % tv * 4;
    float acc[4][4] = {};
    for (int c = 0; c < dk; ++c) {
      float sv[4];
#pragma unroll
      for (int y = 0; y < 4; ++y) sv[y] = j0 + y < dv ? S[(size_t)c * dv + j0 + y] : 0.f;
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const float q = r0 + x < cl ? qs[(r0 + x) * kp + c] : 0.f;
#pragma unroll
        for (int y = 0; y < 4; ++y) acc[x][y] = fmaf(q, sv[y], acc[x][y]);
      }
    }
    for (int s = 0; s < min(cl, r0 + 4); ++s) {
      const float4 v4 = *reinterpret_cast<const float4 *>(vs + s * dvp + j0);
      const float vv[4] = {v4.x, v4.y, v4.z, v4.w};
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const float p = r0 + x < cl ? A[(r0 + x) * C + s] : 0.f;
#pragma unroll
        for (int y = 0; y < 4; ++y) acc[x][y] = fmaf(p, vv[y], acc[x][y]);
      }
    }
#pragma unroll
    for (int x = 0; x < 4; ++x)
#pragma unroll
      for (int y = 0; y < 4; ++y)
        if (r0 + x < cl) os[(r0 + x) * dvp + j0 + y] = acc[x][y];
  }
  __syncthreads();
  for (int t = warp; t < cl; t += ML_THREADS / WARP) {
    const float inv = 1.f / den[t];
    float ss = 0.f;
    for (int j = lane; j < dv; j += WARP) {
      const float o = os[t * dvp + j] * inv;
      ss = fmaf(o, o, ss);
    }
    ss = warp_sum(ss);
    const float r = inv / sqrtf(ss / (float)dv + a.eps);
    const T *row = rows + (size_t)t * a.ld;
    T *out = static_cast<T *>(a.out) + (((size_t)b * a.n + t0 + t) * a.H + h) * dv;
    for (int j = lane; j < dv; j += WARP)
      out[j] = from_f<T>(os[t * dvp + j] * r * a.norm[h * dv + j] * sigmoid_f(to_f(row[goff + j])));
  }
}

// ---- decode: one token per sequence, projections in fp32 -----------------------------------------------------------
// grid (column blocks, H, B), a cluster over the column blocks of a head (the norm needs all of dv). A block reads,
// updates and writes its (dk, columns) part of S once; every block computes n . q for itself, the first one stores n and
// m after the cluster has met.
constexpr int MD_THREADS = 128;
constexpr int MD_MAX_BLOCKS = 8;
constexpr int MD_ROWS = 8;  // state rows of a thread per batch of loads

template <typename T, int V>
__global__ void __launch_bounds__(MD_THREADS) mlstm_decode_kernel(MlstmArgs a, int cols) {
  extern __shared__ float sm[];
  __shared__ float red[2][MD_THREADS / WARP];
  __shared__ float ss_all[MD_MAX_BLOCKS];
  const int tid = threadIdx.x;
  const int cb = blockIdx.x, h = blockIdx.y, b = blockIdx.z, dk = a.dk, dv = a.dv, nb = gridDim.x;
  const int j0 = cb * cols, jn = max(0, min(cols, dv - j0));
  float *q = sm, *k = q + dk, *nn = k + dk, *osum = nn + dk;  // osum: [row groups][cols]
  cg::cluster_group cluster = cg::this_cluster();
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  if (nb > 1) cluster.barrier_arrive();  // (waited for before the first access to another block's memory)
  const float bi = a.bias_i[h], bf = a.bias_f[h];
  asm volatile("griddepcontrol.wait;" ::: "memory");
  const float *row = static_cast<const float *>(a.proj) + (size_t)b * a.ld;
  const float *v = row + 2 * a.H * dk + h * dv + j0, *gate = v + a.H * dv;
  const bool fresh = a.pos[b] == 0;
  float *st = a.state + ((size_t)b * a.H + h) * mlstm_state_stride(dk, dv);
  float *S = st + j0, *N = st + (size_t)dk * dv;
  const int groups = jn / V;                                  // column groups (V divides cols and dv)
  const int rows = max(1, MD_THREADS / max(1, groups));       // row groups
  const int cg0 = tid % max(1, groups) * V, r = tid / max(1, groups);
  const bool mine = r < rows && groups > 0;
  float sr[MD_ROWS][V];
  auto fetch = [&](int c0) {
#pragma unroll
    for (int x = 0; x < MD_ROWS; ++x) {
      const int c = c0 + x * rows;
      const bool ok = mine && c < dk && !fresh;
      const float *p = S + (size_t)c * dv + cg0;
      if (V == 4) {
        float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
        if (ok) t = *reinterpret_cast<const float4 *>(p);
        sr[x][0] = t.x; sr[x][1 % V] = t.y; sr[x][2 % V] = t.z; sr[x][3 % V] = t.w;
      } else {
        sr[x][0] = ok ? p[0] : 0.f;
      }
    }
  };
  fetch(r);
  const float *g = a.gates + (size_t)b * a.ldg + h;
  const float gi = softcap_f(g[0] + bi, a.cap), gf = log_sigmoid_f(softcap_f(g[a.H] + bf, a.cap));
  const float m_old = fresh ? 0.f : N[dk];
  const float m = fmaxf(gf + m_old, gi), keep = expf(gf + m_old - m), add = expf(gi - m);
  float nq = 0.f;
  for (int c = tid; c < dk; c += MD_THREADS) {
    const float qc = row[h * dk + c] * a.scale, kc = add * row[a.H * dk + h * dk + c];
    const float nc = fmaf(keep, fresh ? 0.f : N[c], kc);
    q[c] = qc;
    k[c] = kc;
    nn[c] = nc;
    nq = fmaf(nc, qc, nq);
  }
  nq = warp_sum(nq);
  if (tid % WARP == 0) red[0][tid / WARP] = nq;
  float vv[V], acc[V];
#pragma unroll
  for (int e = 0; e < V; ++e) {
    vv[e] = mine ? v[cg0 + e] : 0.f;
    acc[e] = 0.f;
  }
  __syncthreads();
  for (int c0 = r; c0 < dk; c0 += MD_ROWS * rows) {
    if (c0 != r) fetch(c0);
#pragma unroll
    for (int x = 0; x < MD_ROWS; ++x) {
      const int c = c0 + x * rows;
      if (!mine || c >= dk) continue;
      float *p = S + (size_t)c * dv + cg0;
#pragma unroll
      for (int e = 0; e < V; ++e) {
        sr[x][e] = fmaf(k[c], vv[e], keep * sr[x][e]);
        acc[e] = fmaf(q[c], sr[x][e], acc[e]);
      }
      if (V == 4)
        *reinterpret_cast<float4 *>(p) = make_float4(sr[x][0], sr[x][1 % V], sr[x][2 % V], sr[x][3 % V]);
      else
        p[0] = sr[x][0];
    }
  }
  if (mine) {
#pragma unroll
    for (int e = 0; e < V; ++e) osum[r * cols + cg0 + e] = acc[e];
  }
  __syncthreads();
  nq = 0.f;
#pragma unroll
  for (int x = 0; x < MD_THREADS / WARP; ++x) nq += red[0][x];
  const float inv = 1.f / (fmaxf(fabsf(nq), expf(-m)) + ML_DEN_EPS);
  float ss = 0.f;
  for (int j = tid; j < jn; j += MD_THREADS) {
    float o = 0.f;
    for (int x = 0; x < rows; ++x) o += osum[x * cols + j];
    o *= inv;
    osum[j] = o;  // row group 0's slot of the same column, read by this thread only
    ss = fmaf(o, o, ss);
  }
  ss = warp_sum(ss);
  if (tid % WARP == 0) red[1][tid / WARP] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int x = 0; x < MD_THREADS / WARP; ++x) tot += red[1][x];
  if (nb > 1) {
    cluster.barrier_wait();
    if (tid < nb) cluster.map_shared_rank(ss_all, tid)[cb] = tot;  // this block's sum to every block
    cluster.sync();
    tot = 0.f;
    for (int x = 0; x < nb; ++x) tot += ss_all[x];
  }
  const float rn = 1.f / sqrtf(tot / (float)dv + a.eps);
  T *out = static_cast<T *>(a.out) + ((size_t)b * a.H + h) * dv + j0;
  for (int j = tid; j < jn; j += MD_THREADS)
    out[j] = from_f<T>(osum[j] * rn * a.norm[h * dv + j0 + j] * sigmoid_f(gate[j]));
  if (cb == 0) {  // (all blocks of the head have read the old n and m by now)
    for (int c = tid; c < dk; c += MD_THREADS) N[c] = nn[c];
    if (tid == 0) N[dk] = m;
  }
}

// ---- host ----------------------------------------------------------------------------------------------------------
static size_t state_smem(int C, int dk, int dv) { return 4 * (size_t)C * (up4(dk) + up4(dv)); }
static size_t out_smem(int C, int dk, int dv) {
  return 4 * ((size_t)2 * C * (dk | 1) + (size_t)C * C + 4 + (size_t)2 * C * up4(dv));
}
constexpr size_t ML_SMEM = 220 * 1024;
// chunk length: as long as both kernels' tiles fit into shared memory, 0 if the heads are too large
static int chunk_len(int dk, int dv) {
  for (int C = 64; C >= 8; C /= 2)
    if (state_smem(C, dk, dv) <= ML_SMEM && out_smem(C, dk, dv) <= ML_SMEM) return C;
  return 0;
}
static size_t al256(size_t v) { return (v + 255) / 256 * 256; }

// the tensor-core chunk kernels also need rows that 16-byte copies can read
static bool use_tc(int dtype, const MlstmArgs &a) {
  return mlstm_tc_supported(dtype, a.dk, a.dv) && a.ld % 8 == 0 && aligned16(a.proj) && aligned16(a.out) &&
         aligned16(a.norm);
}

template <typename T>
static int launch_prefill(const MlstmArgs &a, bool tc, cudaStream_t st) {
  const dim3 grid(a.nc, a.H, a.B);
  int rc = DJV_OK;
  if (tc) {
    rc = mlstm_tc_gates(a, st);
    if (rc) return rc;
    rc = mlstm_tc_chunk_state(a, st);
    if (rc) return rc;
  } else {
    cudaFuncSetAttribute(mlstm_chunk_state_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ML_SMEM);
    djv::launch_kernel(mlstm_chunk_state_kernel<T>, grid, dim3(ML_THREADS), state_smem(a.C, a.dk, a.dv), st, a);
    count_launch();
  }
  const int all = a.dk * a.dv + a.dk;
  const bool vec = a.dk % 4 == 0 && a.dv % 4 == 0 && aligned16(a.state);
  const dim3 sg(ceil_div(all, (vec ? 4 : 1) * ML_THREADS), a.H, a.B);
  if (vec && tc) djv::launch_kernel(mlstm_scan_kernel<4, true>, sg, dim3(ML_THREADS), 0, st, a);
  else if (vec) djv::launch_kernel(mlstm_scan_kernel<4, false>, sg, dim3(ML_THREADS), 0, st, a);
  else if (tc) djv::launch_kernel(mlstm_scan_kernel<1, true>, sg, dim3(ML_THREADS), 0, st, a);
  else djv::launch_kernel(mlstm_scan_kernel<1, false>, sg, dim3(ML_THREADS), 0, st, a);
  djv::launch_kernel(mlstm_finish_kernel, dim3(ceil_div(a.B * a.H, 128)), dim3(128), 0, st, a);
  count_launch(2);
  if (tc) return mlstm_tc_chunk_out(a, st);
  cudaFuncSetAttribute(mlstm_chunk_out_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ML_SMEM);
  djv::launch_kernel(mlstm_chunk_out_kernel<T>, grid, dim3(ML_THREADS), out_smem(a.C, a.dk, a.dv), st, a);
  count_launch();
  return check_launch("mlstm_prefill");
}

template <typename T>
static int launch_mlstm_decode(const MlstmArgs &a, cudaStream_t st) {
  const bool vec = a.dv % 4 == 0 && aligned16(a.state);
  const int V = vec ? 4 : 1;
  int nb = 1;  // column blocks: at least 16 columns each
  while (nb < MD_MAX_BLOCKS && a.dv >= 32 * nb) nb *= 2;
  const int cols = ceil_div(ceil_div(a.dv, nb), V) * V;
  nb = ceil_div(a.dv, cols);
  // row groups of a block; the last block may have fewer columns, hence more row groups of them
  auto row_groups = [&](int c) {
    const int g = c / V > 0 ? c / V : 1;
    return MD_THREADS / g > 1 ? MD_THREADS / g : 1;
  };
  const int full = row_groups(cols), last = row_groups(a.dv - (nb - 1) * cols);
  const size_t osum = (size_t)(full > last ? full : last) * cols;
  const size_t smem = 4 * ((size_t)a.dk * 3 + osum);
  DJV_REQUIRE(smem <= 200 * 1024, "mlstm_decode: head sizes %d / %d are too large", a.dk, a.dv);
  const dim3 grid(nb, a.H, a.B), cluster(nb, 1, 1);
  if (vec) {
    cudaFuncSetAttribute(mlstm_decode_kernel<T, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    djv::launch_kernel_cluster(mlstm_decode_kernel<T, 4>, grid, dim3(MD_THREADS), smem, st, cluster, a, cols);
  } else {
    cudaFuncSetAttribute(mlstm_decode_kernel<T, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    djv::launch_kernel_cluster(mlstm_decode_kernel<T, 1>, grid, dim3(MD_THREADS), smem, st, cluster, a, cols);
  }
  count_launch();
  return check_launch("mlstm_decode");
}

}  // namespace djv

using namespace djv;

static int check_mlstm(const char *op, int dtype, const MlstmArgs &a) {
  DJV_REQUIRE(dtype == DJV_DTYPE_BF16 || dtype == DJV_DTYPE_F32, "%s: dtype %d", op, dtype);
  DJV_REQUIRE(a.out && a.proj && a.gates && a.bias_i && a.bias_f && a.norm && a.state && a.pos, "%s: null pointer", op);
  DJV_REQUIRE(a.B >= 1 && a.B <= 65535 && a.n >= 1 && a.H >= 1 && a.H <= 65535, "%s: B=%d n=%d H=%d", op, a.B, a.n, a.H);
  DJV_REQUIRE(a.dk >= 1 && a.dv >= 1 && a.dk <= 1024 && a.dv <= 1024, "%s: head sizes %d / %d", op, a.dk, a.dv);
  DJV_REQUIRE(a.ld >= 2ll * a.H * (a.dk + a.dv) && a.ldg >= 2ll * a.H, "%s: row strides %lld / %lld are too small", op,
              a.ld, a.ldg);
  DJV_REQUIRE(a.cap > 0.f, "%s: gate cap %g", op, (double)a.cap);
  return DJV_OK;
}

extern "C" int djv_mlstm_state_floats(int dk, int dv) { return mlstm_state_stride(dk, dv); }

static int pick_chunk(int dtype, int dk, int dv, bool tc) {
  return tc && mlstm_tc_supported(dtype, dk, dv) ? MLSTM_TC_CHUNK : chunk_len(dk, dv);
}

// scratch of the form that needs more
extern "C" size_t djv_mlstm_scratch_bytes(int dtype, int B, int n, int H, int dk, int dv) {
  if (B < 1 || n < 1 || H < 1 || dk < 1 || dv < 1) return 0;
  size_t most = 0;
  for (int tc = 0; tc < 2; ++tc) {
    const int C = pick_chunk(dtype, dk, dv, tc);
    if (C == 0) continue;
    const size_t rows = (size_t)B * H * ceil_div(n, C);
    size_t need = al256(rows * mlstm_contrib_stride(dk, dv) * 4) + al256(rows * 3 * 8);
    if (tc) need += 2 * al256(rows * dk * dv * 2) + 3 * al256(rows * C * 8);
    if (need > most) most = need;
  }
  return most;
}

extern "C" int djv_mlstm_prefill(int dtype, void *out, const void *proj, long long ld, const float *gates, long long ldg,
                                 const float *bias_i, const float *bias_f, float cap, const float *norm, float eps,
                                 float scale, float *state, const long long *pos, int B, int n, int H, int dk, int dv,
                                 void *scratch, size_t scratch_bytes, void *stream) {
  MlstmArgs a{out, proj, ld, gates, ldg, bias_i, bias_f, cap, norm, eps, scale, state, pos, B, n, H, dk, dv, 0, 0,
              nullptr, nullptr, nullptr, nullptr, nullptr, nullptr, nullptr};
  int rc = check_mlstm("mlstm_prefill", dtype, a);
  if (rc) return rc;
  const bool tc = use_tc(dtype, a);
  a.C = pick_chunk(dtype, dk, dv, tc);
  if (a.C == 0) {
    set_error("mlstm_prefill: head sizes %d / %d are too large", dk, dv);
    return DJV_ERR_UNSUPPORTED;
  }
  a.nc = ceil_div(n, a.C);
  const size_t need = djv_mlstm_scratch_bytes(dtype, B, n, H, dk, dv);
  if (!scratch || scratch_bytes < need || !aligned16(scratch)) {
    set_error("mlstm_prefill: scratch needs %zu bytes (got %zu)", need, scratch_bytes);
    return DJV_ERR_SCRATCH;
  }
  char *p = static_cast<char *>(scratch);
  const size_t rows = (size_t)B * H * a.nc;
  a.contrib = reinterpret_cast<float *>(p);
  p += al256(rows * mlstm_contrib_stride(dk, dv) * 4);
  a.chunk = reinterpret_cast<double *>(p);
  p += al256(rows * 3 * 8);
  if (tc) {
    a.s_hi = reinterpret_cast<bf16 *>(p);
    p += al256(rows * dk * dv * 2);
    a.s_lo = reinterpret_cast<bf16 *>(p);
    p += al256(rows * dk * dv * 2);
    a.g_a = reinterpret_cast<float2 *>(p);
    p += al256(rows * a.C * 8);
    a.g_run = reinterpret_cast<double *>(p);
    p += al256(rows * a.C * 8);
    a.g_sum = reinterpret_cast<double *>(p);
  }
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return dtype == DJV_DTYPE_BF16 ? launch_prefill<bf16>(a, tc, st) : launch_prefill<float>(a, false, st);
}

extern "C" int djv_mlstm_decode(int dtype, void *out, const float *proj, long long ld, const float *gates, long long ldg,
                                const float *bias_i, const float *bias_f, float cap, const float *norm, float eps,
                                float scale, float *state, const long long *pos, int B, int H, int dk, int dv,
                                void *stream) {
  const MlstmArgs a{out, proj, ld, gates, ldg, bias_i, bias_f, cap, norm, eps, scale, state, pos, B, 1, H, dk, dv, 0, 0,
                    nullptr, nullptr, nullptr, nullptr, nullptr, nullptr, nullptr};
  int rc = check_mlstm("mlstm_decode", dtype, a);
  if (rc) return rc;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return dtype == DJV_DTYPE_BF16 ? launch_mlstm_decode<bf16>(a, st) : launch_mlstm_decode<float>(a, st);
}
