// Grouped matrix product of a routed feed-forward on the 5th-generation tensor cores (bf16): rows sorted by expert times
// the experts' weights, with the row weights and the gated unit on the way out.
//
// Persistent blocks, one per multiprocessor, walk output tiles of 128 rows x BN columns; a tile never spans two experts (the
// rows of the next one that a tile's load brings along are not stored). Roles: one thread issues TMA loads into a ring of
// stages, one thread issues the products into one of two accumulators in TMEM, four warps store the other one. Tiles of one
// expert that share weight columns are neighbours, so they meet in L2.
#include <cuda.h>

#include "../../include/dejavu_b200_routed.h"
#include "hybrid_moe.cuh"
#include "tcgen05.cuh"

namespace djv {

constexpr int MG_THREADS = 192, MG_EPI = 128;   // warps 0-3: results; warp 4: loads; warp 5: products
constexpr int MG_M = 128, MG_K = 64;            // rows of a tile, reduction elements of a stage (128 bytes)
constexpr int MG_MAX_EXPERTS = 1024;

__device__ unsigned g_moe_timeouts;  // bounded waits that ran out (never, in a healthy run)

__device__ __forceinline__ void mbar_arrive(uint64_t *bar) {
  asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(bar)) : "memory");
}
// a box of the tensor map at (element x, row y) into this block's shared memory
__device__ __forceinline__ void tma_load_2d(uint32_t dst, const CUtensorMap *map, int x, int y, uint64_t *bar) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(dst),
      "l"(map), "r"(x), "r"(y), "r"(smem_u32(bar))
      : "memory");
}

struct MoeTile {
  int row, rows, wrow, col;  // first row of x, rows that count, first row of the weight matrix, first column of y
};

template <int BN, int STAGES>
__global__ void __launch_bounds__(MG_THREADS, 1)
moe_grouped_tc_kernel(const __grid_constant__ CUtensorMap map_x, const __grid_constant__ CUtensorMap map_w, GroupedArgs a) {
  extern __shared__ unsigned char smem_raw[];
  __shared__ __align__(8) uint64_t full[STAGES], empty[STAGES], acc_full[2], acc_empty[2];
  __shared__ uint32_t tmem_slot;
  __shared__ int offs[MG_MAX_EXPERTS + 1], first[MG_MAX_EXPERTS + 1];  // first row, first row tile of every expert
  constexpr uint32_t A_BYTES = MG_M * 128, B_BYTES = BN * 128;
  const int tid = threadIdx.x, warp = tid / WARP, lane = tid % WARP;
  unsigned char *base = reinterpret_cast<unsigned char *>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const uint32_t ring = smem_u32(base);
  if (tid == 0) {
    for (int s = 0; s < STAGES; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    for (int s = 0; s < 2; ++s) {
      mbar_init(&acc_full[s], 1);
      mbar_init(&acc_empty[s], MG_EPI);
    }
    mbar_fence_init();
  }
  __syncwarp();
  if (warp == 5) tmem_alloc(&tmem_slot, 2 * BN);
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  if (warp == 0) {
    int run = 0;
    for (int e0 = 0; e0 < a.E; e0 += WARP) {
      const int e = e0 + lane, lo = e < a.E ? a.offsets[e] : 0, hi = e < a.E ? a.offsets[e + 1] : 0;
      const int t = (hi - lo + MG_M - 1) / MG_M;
      int s = t;
#pragma unroll
      for (int o = 1; o < WARP; o <<= 1) {
        const int up = __shfl_up_sync(0xffffffffu, s, o);
        if (lane >= o) s += up;
      }
      if (e < a.E) {
        offs[e] = lo;
        first[e] = run + s - t;
      }
      run += __shfl_sync(0xffffffffu, s, WARP - 1);
    }
    if (lane == 0) {
      offs[a.E] = a.offsets[a.E];
      first[a.E] = run;
    }
  }
  __syncthreads();
  tmem_fence_after();
  const uint32_t tm = tmem_slot;
  const int nt = (a.N + BN - 1) / BN, total = first[a.E] * nt, kb = (a.K + MG_K - 1) / MG_K;
  auto locate = [&](int t) {
    int lo = 0, hi = a.E;  // the last expert whose first tile is not after t
    while (hi - lo > 1) {
      const int mid = (lo + hi) / 2;
      if (first[mid] * nt <= t) lo = mid;
      else hi = mid;
    }
    const int mt = first[lo + 1] - first[lo], local = t - first[lo] * nt;
    const int col = local / mt * BN, row = offs[lo] + local % mt * MG_M;
    return MoeTile{row, min(MG_M, offs[lo + 1] - row), lo * a.N + col, col};
  };
  bool dead = false;  // a wait ran out: this role stops, the others run out too
  if (warp == 4 && lane == 0) {
    int it = 0;
    for (int t = blockIdx.x; t < total && !dead; t += gridDim.x) {
      const MoeTile w = locate(t);
      for (int k = 0; k < kb; ++k, ++it) {
        const int s = it % STAGES;
        if (it >= STAGES && !mbar_wait(&empty[s], (it / STAGES - 1) & 1)) {
          dead = true;
          break;
        }
        const uint32_t dst = ring + s * (A_BYTES + B_BYTES);
        mbar_arrive_expect_tx(&full[s], A_BYTES + B_BYTES);
        tma_load_2d(dst, &map_x, k * MG_K, w.row, &full[s]);
        tma_load_2d(dst + A_BYTES, &map_w, k * MG_K, w.wrow, &full[s]);
      }
    }
    if (dead)  // the copies in flight still land
      for (int s = it < STAGES ? 0 : it - STAGES; s < it; ++s) mbar_wait(&full[s % STAGES], (s / STAGES) & 1);
  } else if (warp == 5 && lane == 0) {
    const uint32_t idesc = mma_idesc(MG_M, BN, false, false);
    int it = 0, i = 0;
    for (int t = blockIdx.x; t < total && !dead; t += gridDim.x, ++i) {
      const int acc = i & 1;
      if (i >= 2 && !mbar_wait(&acc_empty[acc], (i / 2 - 1) & 1)) {
        dead = true;
        break;
      }
      tmem_fence_after();
      for (int k = 0; k < kb; ++k, ++it) {
        const int s = it % STAGES;
        if (!mbar_wait(&full[s], (it / STAGES) & 1)) {
          dead = true;
          break;
        }
        tmem_fence_after();
        const uint32_t src = ring + s * (A_BYTES + B_BYTES);
        const uint64_t ad = desc_k_major(src, MG_M, 0), bd = desc_k_major(src + A_BYTES, BN, 0);
#pragma unroll
        for (int x = 0; x < MG_K / 16; ++x) mma_ss(tm + acc * BN, ad + x * 2, bd + x * 2, idesc, k + x > 0);
        mma_commit(&empty[s]);
      }
      if (!dead) mma_commit(&acc_full[acc]);
    }
  } else if (warp < 4) {
    const uint32_t lane_base = (uint32_t)(warp * 32) << 16;
    int i = 0;
    for (int t = blockIdx.x; t < total && !dead; t += gridDim.x, ++i) {
      const MoeTile w = locate(t);
      const int acc = i & 1;
      const bool mine = tid < w.rows;
      const size_t row = (size_t)w.row + tid;
      const float scale = a.scale && mine ? a.scale[row] : 1.f;
      dead = !mbar_wait(&acc_full[acc], (i / 2) & 1);
      dead = __any_sync(0xffffffffu, dead);
      if (dead) break;
      tmem_fence_after();
      bf16 *y = static_cast<bf16 *>(a.y) + row * (a.glu ? a.N / 2 : a.N) + (a.glu ? w.col / 2 : w.col);
#pragma unroll 2
      for (int c = 0; c < BN; c += 32) {
        uint32_t v[32];
        __syncwarp();  // (TMEM accesses are whole-warp instructions)
        tmem_ld32(v, tm + acc * BN + lane_base + c);
        tmem_wait_ld();
        if (!mine) continue;
        if (a.glu) {
#pragma unroll
          for (int e = 0; e < 32; e += 16) {
            if (w.col + c + e < a.N) {  // (N % 16 == 0)
              uint32_t o[4];
#pragma unroll
              for (int x = 0; x < 4; ++x) {
                float u[2];
#pragma unroll
                for (int z = 0; z < 2; ++z) {
                  const float g = scale * __uint_as_float(v[e + 4 * x + 2 * z]);
                  u[z] = __fdividef(g, 1.f + __expf(-g)) * scale * __uint_as_float(v[e + 4 * x + 2 * z + 1]);
                }
                o[x] = pack_bf16(u[0], u[1]);
              }
              *reinterpret_cast<uint4 *>(y + (c + e) / 2) = make_uint4(o[0], o[1], o[2], o[3]);
            }
          }
        } else {
#pragma unroll
          for (int e = 0; e < 32; e += 8) {
            if (w.col + c + e < a.N) {  // (N % 8 == 0)
              uint32_t o[4];
#pragma unroll
              for (int x = 0; x < 4; ++x)
                o[x] = pack_bf16(scale * __uint_as_float(v[e + 2 * x]), scale * __uint_as_float(v[e + 2 * x + 1]));
              *reinterpret_cast<uint4 *>(y + c + e) = make_uint4(o[0], o[1], o[2], o[3]);
            }
          }
        }
      }
      __syncwarp();
      tmem_fence_before();
      mbar_arrive(&acc_empty[acc]);
    }
  }
  if (dead && lane == 0) atomicAdd(&g_moe_timeouts, 1u);
  __syncwarp();
  tmem_fence_before();
  __syncthreads();
  if (warp == 5) {
    tmem_fence_after();
    tmem_dealloc(tm, 2 * BN);
  }
}

using EncodeTiled = CUresult (*)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *, const cuuint64_t *,
                                 const cuuint64_t *, const cuuint32_t *, const cuuint32_t *, CUtensorMapInterleave,
                                 CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

static EncodeTiled encode_tiled() {
  static const EncodeTiled fn = [] {
    void *p = nullptr;
    cudaDriverEntryPointQueryResult found;
    if (cudaGetDriverEntryPointByVersion("cuTensorMapEncodeTiled", &p, 12000, cudaEnableDefault, &found) != cudaSuccess ||
        found != cudaDriverEntryPointSuccess) {
      cudaGetLastError();
      p = nullptr;
    }
    return reinterpret_cast<EncodeTiled>(p);
  }();
  return fn;
}

// rows x cols of bf16, boxes of 64 columns with the 128-byte swizzle, zeros outside
static bool make_map(CUtensorMap *map, const void *p, size_t rows, size_t cols, int box_rows) {
  const cuuint64_t dims[2] = {cols, rows}, strides[1] = {cols * 2};
  const cuuint32_t box[2] = {MG_K, (cuuint32_t)box_rows}, unit[2] = {1, 1};
  return encode_tiled()(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void *>(p), dims, strides, box, unit,
                        CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                        CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

bool moe_grouped_tc_supported(int dtype, const GroupedArgs &a) {
  return dtype == DJV_DTYPE_BF16 && a.K % 8 == 0 && a.N % (a.glu ? 16 : 8) == 0 && a.E <= MG_MAX_EXPERTS &&
         (long long)a.E * a.N < (1ll << 31) && aligned16(a.x) && aligned16(a.w) && aligned16(a.y) && encode_tiled();
}

template <int BN, int STAGES>
static int launch_grouped(const GroupedArgs &a, cudaStream_t st) {
  CUtensorMap mx, mw;
  if (!make_map(&mx, a.x, a.R, a.K, MG_M) || !make_map(&mw, a.w, (size_t)a.E * a.N, a.K, BN)) {
    set_error("moe_grouped: a tensor map was refused");
    return DJV_ERR_CUDA;
  }
  const size_t smem = 1024 + (size_t)STAGES * (MG_M + BN) * 128;
  cudaFuncSetAttribute(moe_grouped_tc_kernel<BN, STAGES>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  const long long tiles = ((long long)a.R / MG_M + a.E) * ceil_div(a.N, BN);  // no fewer than there can be
  const int grid = tiles < sm_count() ? (int)tiles : sm_count();
  djv::launch_kernel(moe_grouped_tc_kernel<BN, STAGES>, dim3(grid), dim3(MG_THREADS), smem, st, mx, mw, a);
  count_launch();
  return check_launch("moe_grouped");
}

int moe_grouped_tc(const GroupedArgs &a, cudaStream_t st) {
  return a.N > 128 ? launch_grouped<256, 4>(a, st) : launch_grouped<128, 6>(a, st);
}

}  // namespace djv

extern "C" unsigned djv_moe_timeouts(void) {
  unsigned v = 0;
  if (cudaMemcpyFromSymbol(&v, djv::g_moe_timeouts, sizeof(v)) != cudaSuccess) {
    cudaGetLastError();
    return 0;
  }
  return v;
}
