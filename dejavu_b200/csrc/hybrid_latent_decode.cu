// Decode attention over latents on the tensor cores (bf16): all heads of a sequence read the same rows, so 16 heads at a
// time are the rows of mma.sync tiles (a decode step has too few rows for the TMEM path's 128).
//
// A block takes 16 heads and a part of the window, 32 tokens per pass:
//   scores: a warp per 8 tokens and half of the row (latent and shared key part);
//   weights: fp32 softmax, two heads per warp, kept as two bf16 terms (hi + lo);
//   sums: a warp takes every 8th group of 16 latent columns of all heads.
// In long parts the next pass's rows load while this one computes. The parts' sums are put together by the kernel that applies the value
// projection.
#include <math.h>

#include "../../include/dejavu_b200_routed.h"
#include "hybrid_latent.cuh"
#include "mma.cuh"

namespace djv {

constexpr int LM_THREADS = 256, LM_WARPS = LM_THREADS / WARP;
constexpr int LM_HEADS = 16, LM_TILE = 32;
constexpr int LM_PP = LM_TILE + 8;  // row pitch of the weights

__host__ __device__ __forceinline__ int lm_pitch(int width) { return ((width + 15) & ~15) + 8; }

template <int NG>  // groups of 16 latent columns per warp
__global__ void __launch_bounds__(LM_THREADS) latent_attend_mma_kernel(LatentDecodeArgs a, int nbuf) {
  extern __shared__ __align__(16) unsigned char sm_raw[];
  __shared__ float sc[2][LM_HEADS][LM_TILE + 4], m_run[LM_HEADS], l_run[LM_HEADS], corr[LM_HEADS];
  __shared__ __align__(16) bf16 p_hi[LM_HEADS * LM_PP], p_lo[LM_HEADS * LM_PP];
  pdl_prologue();
  const int tid = threadIdx.x, lane = tid % WARP, warp = tid / WARP;
  const int h0 = blockIdx.x * LM_HEADS, nh = min(LM_HEADS, a.H - h0), b = blockIdx.y, sp = blockIdx.z;
  const int w = a.rank + a.rot, wp = (w + 15) & ~15, pitch = lm_pitch(w), nch = w / 8;
  bf16 *q = reinterpret_cast<bf16 *>(sm_raw), *tiles = q + LM_HEADS * pitch;
  const bf16 *qr = static_cast<const bf16 *>(a.qc) + ((size_t)b * a.H + h0) * w;
  for (int r = warp; r < LM_HEADS; r += LM_WARPS)
#pragma unroll 3
    for (int c = lane; c < wp / 8; c += WARP) {
      const bool ok = r < nh && c < nch;
      cp_async16_zfill(smem_addr(q + r * pitch + c * 8), ok ? qr + (size_t)r * w + c * 8 : qr, ok ? 16 : 0);
    }
  const long long p = a.pos[b];
  long long lo = p - a.window + 1;
  if (lo < 0) lo = 0;
  const int len = (int)(p - lo + 1), part = (len + a.splits - 1) / a.splits;
  const int t_begin = min(len, sp * part), t_end = min(len, t_begin + part);
  const int slot0 = (int)(lo % a.cap);
  const bf16 *ring = static_cast<const bf16 *>(a.ring) + (size_t)b * a.cap * w;

  auto fetch = [&](int t0, int buf) {
    bf16 *dst = tiles + (size_t)buf * LM_TILE * pitch;
#pragma unroll
    for (int x = 0; x < LM_TILE / LM_WARPS; ++x) {  // a warp per row
      const int r = warp + x * LM_WARPS, t = t0 + r;
      const bool ok = t < t_end;
      int slot = slot0 + t;
      if (slot >= a.cap) slot -= a.cap;
      const bf16 *src = ok ? ring + (size_t)slot * w : ring;
      const uint32_t to = smem_addr(dst + r * pitch);
#pragma unroll 3
      for (int c = lane; c < nch; c += WARP) cp_async16_zfill(to + c * 16, ok ? src + c * 8 : src, ok ? 16 : 0);
    }
    cp_async_commit();
  };
  fetch(t_begin, 0);
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

  const int nt = warp % 4, kh = warp / 4, mid = (wp / 32 + 1) / 2 * 32;  // tokens and part of the row of this warp's scores
  const int k_begin = kh ? min(mid, wp) : 0, k_end = kh ? wp : min(mid, wp);
  int buf = 0;
  for (int t0 = t_begin; t0 < t_end; t0 += LM_TILE) {
    const bool more = t0 + LM_TILE < t_end;
    if (more && nbuf > 1) fetch(t0 + LM_TILE, buf ^ 1);
    if (more && nbuf > 1) cp_async_wait<1>();
    else cp_async_wait<0>();
    __syncthreads();
    const bf16 *tile = tiles + (size_t)buf * LM_TILE * pitch;
    {  // scores of 16 heads against 8 tokens
      float s[4][4] = {};  // independent chains
      const uint32_t qa = smem_addr(q + lrow * pitch + lcol), ka = smem_addr(tile + (nt * 8 + lm) * pitch + lq * 8);
      int k = k_begin;
#pragma unroll 2
      for (; k + 64 <= k_end; k += 64) {
        uint32_t kb[2][4], qf[4][4];
#pragma unroll
        for (int x = 0; x < 2; ++x) ldmatrix_x4(kb[x], ka + k * 2 + x * 64);
#pragma unroll
        for (int x = 0; x < 4; ++x) ldmatrix_x4(qf[x], qa + k * 2 + x * 32);
#pragma unroll
        for (int x = 0; x < 4; ++x)
          mma_m16n8k16_t<bf16>(s[x], qf[x][0], qf[x][1], qf[x][2], qf[x][3], kb[x / 2][x % 2 * 2], kb[x / 2][x % 2 * 2 + 1]);
      }
      for (; k < k_end; k += 16) {
        uint32_t kb[4], qf[4];
        ldmatrix_x4(kb, ka + k * 2);  // (only the first 16 columns are used: the rest may lie past the row)
        ldmatrix_x4(qf, qa + k * 2);
        mma_m16n8k16_t<bf16>(s[0], qf[0], qf[1], qf[2], qf[3], kb[0], kb[1]);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e)
        sc[kh][g + (e / 2) * 8][nt * 8 + t4 * 2 + e % 2] = (s[0][e] + s[1][e]) + (s[2][e] + s[3][e]);
    }
    __syncthreads();
#pragma unroll
    for (int x = 0; x < LM_HEADS / LM_WARPS; ++x) {
      const int r = warp * (LM_HEADS / LM_WARPS) + x;
      const float v = t0 + lane < t_end ? (sc[0][r][lane] + sc[1][r][lane]) * a.scale : -INFINITY;
      const float mx = fmaxf(m_run[r], warp_max(v));
      const float e = expf(v - mx);  // 0 past the end
      const bf16 hi = from_f<bf16>(e);
      p_hi[r * LM_PP + lane] = hi;
      p_lo[r * LM_PP + lane] = from_f<bf16>(e - to_f(hi));
      const float sum = warp_sum(e);
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
        mma_m16n8k16_t<bf16>(acc[x][1], ph[0], ph[1], ph[2], ph[3], v[2], v[3]);
        mma_m16n8k16_t<bf16>(acc[x][0], pl[0], pl[1], pl[2], pl[3], v[0], v[1]);
        mma_m16n8k16_t<bf16>(acc[x][1], pl[0], pl[1], pl[2], pl[3], v[2], v[3]);
      }
    }
    __syncthreads();  // the tile, the scores and the weights are reused
    if (nbuf > 1) buf ^= 1;
    else if (more) fetch(t0 + LM_TILE, 0);
  }
  cp_async_wait<0>();  // (of a part without tokens)
  __syncthreads();
  if (tid < nh) {
    float *ml = a.part_ml + (((size_t)b * a.H + h0 + tid) * a.splits + sp) * 2;
    ml[0] = m_run[tid];
    ml[1] = l_run[tid];
  }
  float *out = a.part_o + (((size_t)b * a.H + h0) * a.splits + sp) * a.rank;
  const size_t step = (size_t)a.splits * a.rank;  // from head to head
#pragma unroll
  for (int x = 0; x < NG; ++x)
#pragma unroll
    for (int y = 0; y < 2; ++y) {
      const int col = (warp + x * LM_WARPS) * 16 + y * 8 + t4 * 2;
      if (col < a.rank) {
        if (g < nh) *reinterpret_cast<float2 *>(out + g * step + col) = make_float2(acc[x][y][0], acc[x][y][1]);
        if (g + 8 < nh) *reinterpret_cast<float2 *>(out + (g + 8) * step + col) = make_float2(acc[x][y][2], acc[x][y][3]);
      }
    }
}

static size_t lm_smem(const LatentDecodeArgs &a, int nbuf) {
  // (32 bytes more: a last step of 16 columns loads 32)
  return (LM_HEADS + (size_t)nbuf * LM_TILE) * lm_pitch(a.rank + a.rot) * 2 + 32;
}
constexpr size_t LM_SMEM = 200 * 1024;

int latent_splits(int B, int H, int window) {
  // at most two blocks of 16 heads per multiprocessor, a pass of tokens each
  const long long groups = (long long)B * ceil_div(H, LM_HEADS);
  long long s = 2 * sm_count() / groups;
  if (s > ceil_div(window, LM_TILE)) s = ceil_div(window, LM_TILE);
  return s < 1 ? 1 : (s > LD_MAX_SPLITS ? LD_MAX_SPLITS : (int)s);
}

bool latent_attend_mma_supported(const LatentDecodeArgs &a, bool bf16_rows) {
  return bf16_rows && a.rank % 8 == 0 && a.rot % 8 == 0 && a.rank <= 1024 && aligned16(a.ring) && aligned16(a.qc) &&
         aligned16(a.part_o) && lm_smem(a, 1) <= LM_SMEM;
}

int latent_attend_mma(const LatentDecodeArgs &a, cudaStream_t st) {
  const int part = ceil_div(a.window, a.splits), nbuf = part > 4 * LM_TILE && lm_smem(a, 2) <= LM_SMEM ? 2 : 1;
  const size_t smem = lm_smem(a, nbuf);
  const dim3 grid(ceil_div(a.H, LM_HEADS), a.B, a.splits);
  // No more shared memory per multiprocessor than the blocks of this launch fill: in a chain of early launched kernels the
  // ones that follow live with the split between shared memory and L1 they find, and they want L1 for their activations.
  const long long blocks = (long long)grid.x * grid.y * grid.z;
  const int per_sm = blocks <= sm_count() ? 1 : 2;
  const int carveout = (int)((per_sm * (smem + 8 * 1024) * 100 + 228 * 1024 - 1) / (228 * 1024));
#define DJV_GO(G_)                                                                                                       \
  {                                                                                                                      \
    cudaFuncSetAttribute(latent_attend_mma_kernel<G_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)LM_SMEM);       \
    cudaFuncSetAttribute(latent_attend_mma_kernel<G_>, cudaFuncAttributePreferredSharedMemoryCarveout,                   \
                         carveout < 100 ? carveout : 100);                                                               \
    djv::launch_kernel(latent_attend_mma_kernel<G_>, grid, dim3(LM_THREADS), smem, st, a, nbuf);                         \
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
