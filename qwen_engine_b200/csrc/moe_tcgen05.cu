// The grouped products of routed experts without a gate for steps of many rows, bfloat16, on tcgen05:
//
//   qe_moe_gather       xs[p, :] = x[sorted_pair[p] / top, :]: the pairs' rows in the experts' order
//   qe_moe_tc           out[p, :] = f(W_e xs[p, :]) for the pairs p of expert e (bfloat16, the first product) or
//                       W_e a[p, :] (float32, the second one)
//
// An expert's rows lie side by side, so a tile of 128 of them is one TMA box wherever it starts (its last tile reads into
// the next expert's rows, which are not stored), and the experts' weights are one matrix of E N rows.  Persistent, one CTA per SM:
// the tiles are numbered expert by expert, and every CTA lays out their numbers from the device's offsets itself, so
// nothing of the launch depends on the routing.  128 x 256 tiles: warp 0 feeds a ring of four stages by TMA (128-byte
// swizzle), one thread of warp 1 issues tcgen05.mma into two accumulators in tensor memory, warps 2 to 5 read one of them
// out while the next tile's products run.  Every wait is bounded.  A row's bits depend on K alone.
#include "tcgen05.cuh"

#define MT_BM 128
#define MT_BN 256
#define MT_BK 64
#define MT_STAGES 4
#define MT_THREADS 192
#define MT_MAX_E 1024

static __device__ int g_tc_status = 0;      // 0 = fine; else code of the first wait that ran out

struct __align__(1024) MtSmem {
  __nv_bfloat16 a[MT_STAGES][MT_BM * MT_BK];          // 16 KB each
  __nv_bfloat16 b[MT_STAGES][MT_BN * MT_BK];          // 32 KB each
  uint64_t full[MT_STAGES];
  uint64_t empty[MT_STAGES];
  uint64_t acc_full[2], acc_empty[2];
  uint32_t tmem_base;
  int abort_flag;
  int tiles_before[MT_MAX_E + 1];                     // row tiles of the experts before e
};

__device__ __forceinline__ int mt_warp_scan(int v, int lane) {      // inclusive
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) { const int u = __shfl_up_sync(0xffffffffu, v, o); if (lane >= o) v += u; }
  return v;
}

// the expert whose row tiles hold number m: the last e with tiles_before[e] <= m
__device__ __forceinline__ int mt_expert_of(const int* tiles_before, int E, int m) {
  int lo = 0, hi = E - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (tiles_before[mid] <= m) lo = mid; else hi = mid - 1;
  }
  return lo;
}

__global__ void __launch_bounds__(128)
moe_gather_kernel(const uint4* __restrict__ x, const int* __restrict__ sorted_pair, uint4* __restrict__ xs, int K8, int top) {
  pdl_launch_dependents();
  pdl_wait();
  const uint4* src = x + (size_t)(__ldg(sorted_pair + blockIdx.x) / top) * K8;
  uint4* dst = xs + (size_t)blockIdx.x * K8;
#pragma unroll 2
  for (int i = threadIdx.x; i < K8; i += 128) dst[i] = src[i];
}

// UP: bfloat16 out = f(sums); else float32 out = sums.  N: weight rows of an expert.
template <bool UP>
__global__ void __launch_bounds__(MT_THREADS, 1)
moe_tcgen05_kernel(const __grid_constant__ CUtensorMap map_x, const __grid_constant__ CUtensorMap map_w,
                   const int* __restrict__ offsets, void* __restrict__ out_, int E, int N, int K, int act) {
  extern __shared__ unsigned char smem_raw[];
  constexpr uint32_t TMEM_COLS = 2 * MT_BN;
  constexpr uint32_t STAGE_BYTES = (MT_BM + MT_BN) * MT_BK * sizeof(__nv_bfloat16);
  pdl_launch_dependents();
  MtSmem& sm = *reinterpret_cast<MtSmem*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int num_kb = (K + MT_BK - 1) / MT_BK;
  const int n_blocks = (N + MT_BN - 1) / MT_BN;
  volatile int* abort_flag = &sm.abort_flag;
  if (threadIdx.x == 0) {
    tma_prefetch_map(&map_x);
    tma_prefetch_map(&map_w);
    for (int s = 0; s < MT_STAGES; ++s) { mbar_init(&sm.full[s], 1); mbar_init(&sm.empty[s], 1); }
    for (int s = 0; s < 2; ++s) { mbar_init(&sm.acc_full[s], 1); mbar_init(&sm.acc_empty[s], 4); }
    sm.abort_flag = 0;
    mbar_init_fence();
  }
  if (warp == 1) tc_alloc(&sm.tmem_base, TMEM_COLS);
  pdl_wait();
  if (warp == 2) {                                    // the tiles' numbers, from the offsets the sort left
    int run = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int e = e0 + lane;
      const int t = e < E ? (__ldcg(offsets + e + 1) - __ldcg(offsets + e) + MT_BM - 1) / MT_BM : 0;
      const int inc = mt_warp_scan(t, lane);
      if (e < E) sm.tiles_before[e] = run + inc - t;
      run += __shfl_sync(0xffffffffu, inc, 31);
    }
    if (lane == 0) sm.tiles_before[E] = run;
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = sm.tmem_base;
  const int n_tiles = sm.tiles_before[E] * n_blocks;
  // tile -> its expert, first sorted row and first weight row (columns vary fastest: a row tile's boxes are used again at once)
  auto tile_at = [&](int tile, int& e, int& first, int& n0) {
    const int m = tile / n_blocks;
    e = mt_expert_of(sm.tiles_before, E, m);
    first = __ldcg(offsets + e) + (m - sm.tiles_before[e]) * MT_BM;
    n0 = (tile - m * n_blocks) * MT_BN;
  };

  if (warp == 0) {
    if (lane == 0) {
      uint32_t kc = 0;
      bool ok = true;
      for (int tile = blockIdx.x; ok && tile < n_tiles; tile += gridDim.x) {
        int e, first, n0;
        tile_at(tile, e, first, n0);
        for (int kb = 0; kb < num_kb; ++kb, ++kc) {
          const uint32_t s = kc % MT_STAGES, round = kc / MT_STAGES;
          if (round > 0 && !mbar_wait(&sm.empty[s], (round - 1) & 1, abort_flag, 41, &g_tc_status)) { ok = false; break; }
          mbar_expect_tx(&sm.full[s], STAGE_BYTES);
          tma_load_2d(sm.a[s], &map_x, &sm.full[s], kb * MT_BK, first);
          tma_load_2d(sm.b[s], &map_w, &sm.full[s], kb * MT_BK, e * N + n0);
        }
      }
      if (!ok) {
        // giving up: let the copies that are still in flight land before the CTA leaves (bounded)
        for (uint32_t i = kc > (uint32_t)MT_STAGES ? kc - MT_STAGES : 0; i < kc; ++i)
          for (uint32_t spin = 0; spin < TC_WAIT_LIMIT; ++spin)
            if (mbar_try_wait(&sm.full[i % MT_STAGES], (i / MT_STAGES) & 1)) break;
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc = make_idesc(MT_BM, MT_BN);
      uint32_t kc = 0;
      bool ok = true;
      int it = 0;
      for (int tile = blockIdx.x; ok && tile < n_tiles; tile += gridDim.x, ++it) {
        const int buf = it & 1;
        if (it >= 2 && !mbar_wait(&sm.acc_empty[buf], ((it >> 1) - 1) & 1, abort_flag, 44, &g_tc_status)) { ok = false; break; }
        tc_fence_after();
        const uint32_t acc = tmem + buf * MT_BN;
        for (int kb = 0; kb < num_kb; ++kb, ++kc) {
          const uint32_t s = kc % MT_STAGES;
          if (!mbar_wait(&sm.full[s], (kc / MT_STAGES) & 1, abort_flag, 42, &g_tc_status)) { ok = false; break; }
          tc_fence_after();
          const uint64_t da = make_smem_desc(smem_u32(sm.a[s]));
          const uint64_t db = make_smem_desc(smem_u32(sm.b[s]));
#pragma unroll
          for (int k = 0; k < MT_BK / 16; ++k) tc_mma_bf16(acc, da + 2 * k, db + 2 * k, idesc, (kb | k) != 0);
          tc_commit(&sm.empty[s]);
        }
        if (ok) tc_commit(&sm.acc_full[buf]);
      }
    }
  } else {
    const int quarter = warp & 3;
    int it = 0;
    for (int tile = blockIdx.x; tile < n_tiles; tile += gridDim.x, ++it) {
      const int buf = it & 1;
      int e, first, n0;
      tile_at(tile, e, first, n0);
      const int rows = __ldcg(offsets + e + 1) - first;           // (may be more than the tile's)
      if (!__all_sync(0xffffffffu, mbar_wait(&sm.acc_full[buf], (it >> 1) & 1, abort_flag, 43, &g_tc_status))) break;
      tc_fence_after();
      const int r = quarter * 32 + lane;
      const bool full8 = (N % 8) == 0;
#pragma unroll 1
      for (int c0 = 0; c0 < MT_BN; c0 += 32) {
        uint32_t v[32];
        tc_ld_32x32b_x32(tmem + ((uint32_t)(quarter * 32) << 16) + buf * MT_BN + c0, v);
        tc_wait_ld();
        if (c0 + 32 == MT_BN) {
          tc_fence_before();
          __syncwarp();
          if (lane == 0) mbar_arrive(&sm.acc_empty[buf]);
        }
        const size_t at = (size_t)(first + r) * N + n0 + c0;
        const bool live = r < rows && n0 + c0 < N;
        if (!live) {
        } else if constexpr (UP) {
          __nv_bfloat16* dst = (__nv_bfloat16*)out_ + at;
#pragma unroll
          for (int j = 0; j < 32; ++j) v[j] = __float_as_uint(act_fast(__uint_as_float(v[j]), act));
          if (full8 && n0 + c0 + 32 <= N) {
#pragma unroll
            for (int j = 0; j < 32; j += 8) {
              uint32_t p[4];
#pragma unroll
              for (int i = 0; i < 4; ++i) {
                __nv_bfloat162 b2 = __floats2bfloat162_rn(__uint_as_float(v[j + 2 * i]), __uint_as_float(v[j + 2 * i + 1]));
                p[i] = *reinterpret_cast<uint32_t*>(&b2);
              }
              *reinterpret_cast<uint4*>(dst + j) = make_uint4(p[0], p[1], p[2], p[3]);
            }
          } else {
#pragma unroll
            for (int j = 0; j < 32; ++j)
              if (n0 + c0 + j < N) dst[j] = __float2bfloat16_rn(__uint_as_float(v[j]));
          }
        } else {
          float* dst = (float*)out_ + at;
          if (full8 && n0 + c0 + 32 <= N) {
#pragma unroll
            for (int j = 0; j < 32; j += 4)
              *reinterpret_cast<float4*>(dst + j) = make_float4(__uint_as_float(v[j]), __uint_as_float(v[j + 1]),
                                                                __uint_as_float(v[j + 2]), __uint_as_float(v[j + 3]));
          } else {
#pragma unroll
            for (int j = 0; j < 32; ++j)
              if (n0 + c0 + j < N) dst[j] = __uint_as_float(v[j]);
          }
        }
        __syncwarp();
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tc_dealloc(tmem, TMEM_COLS);
  }
}

extern "C" int qe_moe_tc_status() {
  int v = 0;
  cudaMemcpyFromSymbol(&v, g_tc_status, sizeof(int));
  return v;
}
extern "C" void qe_moe_tc_clear_status() {
  int v = 0;
  cudaMemcpyToSymbol(g_tc_status, &v, sizeof(int));
}

// xs [P, K] bfloat16; K a multiple of 8
extern "C" int qe_moe_gather(const void* x, const int* sorted_pair, void* xs, int P, int K, int top, cudaStream_t stream) {
  if (P <= 0) return 0;
  if (K < 8 || K % 8 || top < 1 || (((uintptr_t)x | (uintptr_t)xs) & 15)) QE_REFUSE("moe_gather: rows of %d channels", K);
  qe_launch(moe_gather_kernel, dim3(P), dim3(128), 0, stream, (const uint4*)x, sorted_pair, (uint4*)xs, K / 8, top);
  QE_CHECK_LAUNCH("moe_gather");
  return 0;
}

// rows [P, K] in the experts' order, w [E, N, K]; up: out bfloat16 [P, N] = f(product) (act: common.cuh), else float32 [P, N].
extern "C" int qe_moe_tc(const void* rows, const void* w, const int* offsets, void* out, int P, int E, int N, int K, int act, int up,
                         cudaStream_t stream) {
  if (P <= 0) return 0;
  if (K < 8 || K % 8 || E < 1 || E > MT_MAX_E || N < 1) QE_REFUSE("moe_tc: %d experts of %d x %d", E, N, K);
  if ((long)E * N > 0x7fffffffL) QE_REFUSE("moe_tc: %d experts of %d rows", E, N);
  if (act < 0 || act > QE_ACT_MAX || (act && !up)) QE_REFUSE("moe_tc: activation %d", act);
  if (((uintptr_t)rows | (uintptr_t)w | (uintptr_t)out) & 15) QE_REFUSE("moe_tc: operands must be 16-byte aligned");
  CUtensorMap map_x, map_w;
  const uint64_t strides[1] = {(uint64_t)K * 2};
  {
    const uint64_t dims[2] = {(uint64_t)K, (uint64_t)P};
    const uint32_t box[2] = {MT_BK, MT_BM};
    if (!qe_tensor_map_bf16(rows, 2, dims, strides, box, &map_x)) return 1;
  }
  {
    const uint64_t dims[2] = {(uint64_t)K, (uint64_t)E * (uint64_t)N};
    const uint32_t box[2] = {MT_BK, MT_BN};
    if (!qe_tensor_map_bf16(w, 2, dims, strides, box, &map_w)) return 1;
  }
  const size_t smem = sizeof(MtSmem) + 1024;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(moe_tcgen05_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(moe_tcgen05_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) QE_REFUSE("moe_tc: shared memory %zu: %s", smem, cudaGetErrorString(e));
    configured = true;
  }
  static int sms = 0;
  if (sms == 0) {
    int dev = 0, v = 148;
    if (cudaGetDevice(&dev) == cudaSuccess) cudaDeviceGetAttribute(&v, cudaDevAttrMultiProcessorCount, dev);
    sms = v > 0 ? v : 148;
  }
  const long worst = ((long)(P + MT_BM - 1) / MT_BM + (E < P ? E : P)) * ((N + MT_BN - 1) / MT_BN);
  const dim3 grid((unsigned)(worst < sms ? worst : sms));
  if (up) qe_launch(moe_tcgen05_kernel<true>, grid, dim3(MT_THREADS), smem, stream, map_x, map_w, offsets, out, E, N, K, act);
  else qe_launch(moe_tcgen05_kernel<false>, grid, dim3(MT_THREADS), smem, stream, map_x, map_w, offsets, out, E, N, K, 0);
  QE_CHECK_LAUNCH("moe_tc");
  return 0;
}
