// Decode attention over latents on the tensor cores (bf16): all heads of a sequence read the same rows, so 16 heads at a
// time are the rows of mma.sync tiles (a decode step has too few rows for the TMEM path's 128).
//
// A block takes 16 heads and a part of the window, 64 tokens per pass:
//   scores: a warp per 8 tokens, over the whole row (latent and shared key part);
//   weights: fp32 softmax, two heads per warp, kept as two bf16 terms (hi + lo);
//   sums: a warp takes every 8th group of 16 latent columns of all heads.
// The next pass's rows load while this one computes. The parts of a window are a cluster; each of its blocks combines a share
// of the columns from all of them.
#include <cooperative_groups.h>
#include <math.h>

#include "../../include/dejavu_b200_routed.h"
#include "hybrid_latent.cuh"
#include "mma.cuh"

namespace djv {

namespace cg = cooperative_groups;

constexpr int LM_THREADS = 256, LM_WARPS = LM_THREADS / WARP;
constexpr int LM_HEADS = 16, LM_TILE = 64, LM_MAX_SPLITS = 8;
constexpr int LM_PP = LM_TILE + 8;  // row pitch of the weights

__host__ __device__ __forceinline__ int lm_pitch(int width) { return ((width + 15) & ~15) + 8; }

template <int NG>  // groups of 16 latent columns per warp
__global__ void __launch_bounds__(LM_THREADS) latent_attend_mma_kernel(LatentDecodeArgs a, int nbuf) {
  extern __shared__ __align__(16) unsigned char sm_raw[];
  __shared__ __align__(16) float sc[LM_HEADS][LM_TILE + 4], part_m[LM_MAX_SPLITS][LM_HEADS], part_l[LM_MAX_SPLITS][LM_HEADS];
  __shared__ float m_run[LM_HEADS], l_run[LM_HEADS], corr[LM_HEADS];
  __shared__ __align__(16) bf16 p_hi[LM_HEADS * LM_PP], p_lo[LM_HEADS * LM_PP];
  cg::cluster_group cluster = cg::this_cluster();
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  const int nsplit = gridDim.z;
  if (nsplit > 1) cluster.barrier_arrive();  // (waited for before the first access to another block's memory)
  asm volatile("griddepcontrol.wait;" ::: "memory");
  const int tid = threadIdx.x, lane = tid % WARP, warp = tid / WARP;
  const int h0 = blockIdx.x * LM_HEADS, nh = min(LM_HEADS, a.H - h0), b = blockIdx.y, sp = blockIdx.z;
  const int w = a.rank + a.rot, wp = (w + 15) & ~15, pitch = lm_pitch(w), nch = w / 8;
  bf16 *q = reinterpret_cast<bf16 *>(sm_raw), *tiles = q + LM_HEADS * pitch;
  const long long p = a.pos[b];
  long long lo = p - a.window + 1;
  if (lo < 0) lo = 0;
  const int len = (int)(p - lo + 1), part = (len + nsplit - 1) / nsplit;
  const int t_begin = min(len, sp * part), t_end = min(len, t_begin + part);
  const int slot0 = (int)(lo % a.cap);
  const bf16 *ring = static_cast<const bf16 *>(a.ring) + (size_t)b * a.cap * w;

  auto fetch = [&](int t0, int buf) {
    bf16 *dst = tiles + (size_t)buf * LM_TILE * pitch;
    for (int i = tid; i < LM_TILE * nch; i += LM_THREADS) {
      const int r = i / nch, c = i - r * nch, t = t0 + r;
      const bool ok = t < t_end;
      int slot = slot0 + t;
      if (slot >= a.cap) slot -= a.cap;
      cp_async16_zfill(smem_addr(dst + r * pitch + c * 8), ok ? ring + (size_t)slot * w + c * 8 : ring, ok ? 16 : 0);
    }
    cp_async_commit();
  };
  fetch(t_begin, 0);
  const bf16 *qr = static_cast<const bf16 *>(a.qc) + ((size_t)b * a.H + h0) * w;
  for (int i = tid; i < LM_HEADS * wp / 8; i += LM_THREADS) {
    const int r = i / (wp / 8), c = i - r * (wp / 8);
    *reinterpret_cast<uint4 *>(q + r * pitch + c * 8) =
        r < nh && c < nch ? *reinterpret_cast<const uint4 *>(qr + (size_t)r * w + c * 8) : make_uint4(0, 0, 0, 0);
  }
  if (nch * 8 < wp)  // the columns that pad a row to whole tiles
    for (int i = tid; i < nbuf * LM_TILE; i += LM_THREADS)
      *reinterpret_cast<uint4 *>(tiles + (size_t)i * pitch + nch * 8) = make_uint4(0, 0, 0, 0);
  if (tid < LM_HEADS) {
    m_run[tid] = -INFINITY;
    l_run[tid] = 0.f;
  }
  const int g = lane / 4, t4 = lane % 4, lm = lane % 8, lq = lane / 8;
  const int lrow = (lq % 2) * 8 + lm, lcol = (lq / 2) * 8;  // ldmatrix rows of an A operand
  float acc[NG][2][4];
#pragma unroll
  for (int x = 0; x < NG; ++x)
#pragma unroll
    for (int y = 0; y < 2; ++y)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[x][y][e] = 0.f;

  int buf = 0;
  for (int t0 = t_begin; t0 < t_end; t0 += LM_TILE) {
    const bool more = t0 + LM_TILE < t_end;
    if (more && nbuf > 1) fetch(t0 + LM_TILE, buf ^ 1);
    if (more && nbuf > 1) cp_async_wait<1>();
    else cp_async_wait<0>();
    __syncthreads();
    const bf16 *tile = tiles + (size_t)buf * LM_TILE * pitch;
    {  // scores of 16 heads against this warp's 8 tokens
      float s[2][4] = {};
      const uint32_t qa = smem_addr(q + lrow * pitch + lcol), ka = smem_addr(tile + (warp * 8 + lm) * pitch + lq * 8);
      for (int k = 0; k < wp; k += 32) {
        uint32_t kb[4], qf[4];
        ldmatrix_x4(kb, ka + k * 2);  // k .. k+31 (the second half may be past the row: the pitch's pad, not used)
        ldmatrix_x4(qf, qa + k * 2);
        mma_m16n8k16_t<bf16>(s[0], qf[0], qf[1], qf[2], qf[3], kb[0], kb[1]);
        if (k + 16 < wp) {
          ldmatrix_x4(qf, qa + k * 2 + 32);
          mma_m16n8k16_t<bf16>(s[1], qf[0], qf[1], qf[2], qf[3], kb[2], kb[3]);
        }
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = warp * 8 + t4 * 2 + e % 2;
        sc[g + (e / 2) * 8][t] = t0 + t < t_end ? (s[0][e] + s[1][e]) * a.scale : -INFINITY;
      }
    }
    __syncthreads();
#pragma unroll
    for (int x = 0; x < LM_HEADS / LM_WARPS; ++x) {
      const int r = warp * (LM_HEADS / LM_WARPS) + x;
      const float2 v = *reinterpret_cast<const float2 *>(&sc[r][lane * 2]);
      const float mx = fmaxf(m_run[r], warp_max(fmaxf(v.x, v.y)));
      const float e0 = expf(v.x - mx), e1 = expf(v.y - mx);  // 0 past the end
      const uint32_t hi = pack_bf16(e0, e1);
      const float2 top = b2f(hi);
      *reinterpret_cast<uint32_t *>(p_hi + r * LM_PP + lane * 2) = hi;
      *reinterpret_cast<uint32_t *>(p_lo + r * LM_PP + lane * 2) = pack_bf16(e0 - top.x, e1 - top.y);
      const float sum = warp_sum(e0 + e1);
      __syncwarp();
      if (lane == 0) {
        corr[r] = m_run[r] == -INFINITY ? 0.f : expf(m_run[r] - mx);
        l_run[r] = l_run[r] * corr[r] + sum;
        m_run[r] = mx;
      }
    }
    __syncthreads();
    const float c0 = corr[g], c1 = corr[g + 8];
#pragma unroll
    for (int x = 0; x < NG; ++x)
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        acc[x][y][0] *= c0;
        acc[x][y][1] *= c0;
        acc[x][y][2] *= c1;
        acc[x][y][3] *= c1;
      }
#pragma unroll
    for (int k = 0; k < LM_TILE; k += 16) {
      uint32_t ph[4], pl[4];
      ldmatrix_x4(ph, smem_addr(p_hi + lrow * LM_PP + k + lcol));
      ldmatrix_x4(pl, smem_addr(p_lo + lrow * LM_PP + k + lcol));
#pragma unroll
      for (int x = 0; x < NG; ++x) {
        const int col = (warp + x * LM_WARPS) * 16;
        if (col >= a.rank) continue;  // (rank % 8 == 0; a half group past the latents reads the row's next columns)
        uint32_t v[4];  // (t 0-7, c 0-7), (t 8-15, c 0-7), (t 0-7, c 8-15), (t 8-15, c 8-15)
        ldmatrix_x4_trans(v, smem_addr(tile + (k + (lq % 2) * 8 + lm) * pitch + col + (lq / 2) * 8));
        mma_m16n8k16_t<bf16>(acc[x][0], ph[0], ph[1], ph[2], ph[3], v[0], v[1]);
        mma_m16n8k16_t<bf16>(acc[x][0], pl[0], pl[1], pl[2], pl[3], v[0], v[1]);
        mma_m16n8k16_t<bf16>(acc[x][1], ph[0], ph[1], ph[2], ph[3], v[2], v[3]);
        mma_m16n8k16_t<bf16>(acc[x][1], pl[0], pl[1], pl[2], pl[3], v[2], v[3]);
      }
    }
    __syncthreads();  // the tile, the scores and the weights are reused
    if (nbuf > 1) buf ^= 1;
    else if (more) fetch(t0 + LM_TILE, 0);
  }
  cp_async_wait<0>();  // (of a part without tokens)
  __syncthreads();
  float *part_o = reinterpret_cast<float *>(sm_raw);  // [heads][rank]: over the queries and tiles
  const int op = a.rank;
#pragma unroll
  for (int x = 0; x < NG; ++x)
#pragma unroll
    for (int y = 0; y < 2; ++y) {
      const int col = (warp + x * LM_WARPS) * 16 + y * 8 + t4 * 2;
      if (col < a.rank) {
        *reinterpret_cast<float2 *>(part_o + g * op + col) = make_float2(acc[x][y][0], acc[x][y][1]);
        *reinterpret_cast<float2 *>(part_o + (g + 8) * op + col) = make_float2(acc[x][y][2], acc[x][y][3]);
      }
    }
  if (nsplit > 1) {
    cluster.barrier_wait();
    cluster.sync();  // every block's sums are in place
  } else {
    __syncthreads();
  }
  // factors of the parts, then this block's share of the columns
  if (tid < nsplit * LM_HEADS) {
    const int s = tid / LM_HEADS, r = tid % LM_HEADS;
    part_m[s][r] = nsplit > 1 ? cluster.map_shared_rank(m_run, s)[r] : m_run[r];
    part_l[s][r] = nsplit > 1 ? cluster.map_shared_rank(l_run, s)[r] : l_run[r];
  }
  __syncthreads();
  if (tid < LM_HEADS) {
    float m = -INFINITY, l = 0.f;
    for (int s = 0; s < nsplit; ++s) m = fmaxf(m, part_m[s][tid]);
    for (int s = 0; s < nsplit; ++s) {
      const float f = part_m[s][tid] == -INFINITY ? 0.f : expf(part_m[s][tid] - m);
      l = fmaf(f, part_l[s][tid], l);
      part_m[s][tid] = f;
    }
    for (int s = 0; s < nsplit; ++s) part_m[s][tid] /= l;
  }
  __syncthreads();
  const int share = ((a.rank + nsplit - 1) / nsplit + 1) & ~1, j0 = min(a.rank, sp * share), jn = min(share, a.rank - j0) / 2;
  float *out = a.ctx + ((size_t)b * a.H + h0) * a.rank;
  for (int i = tid; i < nh * jn; i += LM_THREADS) {
    const int r = i / jn, j = j0 + (i - r * jn) * 2;
    float2 v[LM_MAX_SPLITS];
#pragma unroll
    for (int s = 0; s < LM_MAX_SPLITS; ++s)
      if (s < nsplit)
        v[s] = *reinterpret_cast<const float2 *>((nsplit > 1 ? cluster.map_shared_rank(part_o, s) : part_o) + r * op + j);
    float2 o = make_float2(0.f, 0.f);
#pragma unroll
    for (int s = 0; s < LM_MAX_SPLITS; ++s)
      if (s < nsplit) {
        o.x = fmaf(part_m[s][r], v[s].x, o.x);
        o.y = fmaf(part_m[s][r], v[s].y, o.y);
      }
    *reinterpret_cast<float2 *>(out + (size_t)r * a.rank + j) = o;
  }
  if (nsplit > 1) cluster.sync();  // no block leaves while another may still read its sums
}

static size_t lm_smem(const LatentDecodeArgs &a, int nbuf) {
  const size_t pitch = lm_pitch(a.rank + a.rot);
  // (32 bytes more: the last row's second half of a 32-column step)
  const size_t work = (LM_HEADS + (size_t)nbuf * LM_TILE) * pitch * 2 + 32, sums = (size_t)LM_HEADS * a.rank * 4;
  return work > sums ? work : sums;
}
constexpr size_t LM_SMEM = 210 * 1024;

bool latent_attend_mma_supported(const LatentDecodeArgs &a, bool bf16_rows) {
  return bf16_rows && a.rank % 8 == 0 && a.rot % 8 == 0 && a.rank <= 1024 && aligned16(a.ring) && aligned16(a.qc) &&
         lm_smem(a, 1) <= LM_SMEM;
}

int latent_attend_mma(const LatentDecodeArgs &a, cudaStream_t st) {
  const int nbuf = lm_smem(a, 2) <= LM_SMEM ? 2 : 1;
  const size_t smem = lm_smem(a, nbuf);
  const int hb = ceil_div(a.H, LM_HEADS);
  // parts of the window: as long as each has a pass of its own and the blocks fit the device at once
  int nsplit = 1;
  while (nsplit < LM_MAX_SPLITS && a.window > LM_TILE * nsplit && (long long)hb * a.B * nsplit * 2 <= sm_count()) nsplit *= 2;
  const dim3 grid(hb, a.B, nsplit);
#define DJV_GO(G_)                                                                                                       \
  {                                                                                                                      \
    cudaFuncSetAttribute(latent_attend_mma_kernel<G_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)LM_SMEM);       \
    djv::launch_kernel_cluster(latent_attend_mma_kernel<G_>, grid, dim3(LM_THREADS), smem, st, dim3(1, 1, nsplit), a,    \
                               nbuf);                                                                                    \
  }
  const int ng = ceil_div(a.rank, 16 * LM_WARPS);
  if (ng == 1) DJV_GO(1)
  else if (ng == 2) DJV_GO(2)
  else if (ng <= 4) DJV_GO(4)
  else DJV_GO(8)
#undef DJV_GO
  count_launch();
  return check_launch("latent_decode");
}

}  // namespace djv
