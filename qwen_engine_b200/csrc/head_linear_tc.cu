// out[t, h, :N] = W[h] x[t, h, :K] for many rows in bfloat16 on tcgen05: the products with one matrix per head around the
// attention over a latent cache (latent_attention.cu), optionally times sigmoid(gate[t, h]) before the rounding.
//
// The rows are a three-dimensional tensor (channel, head, token) whatever their strides, so a tile's operand is one TMA box
// per 64 channels that ends with the head (zero fill beyond K).  Persistent, one CTA per SM over the tiles of 128 tokens x
// BN columns of a head (BN 64, 128, 192 or 256 by N): warp 0 feeds a ring of stages, one thread of warp 1 issues tcgen05.mma
// into two accumulators in tensor memory, warps 2 to 9 (two per quarter of the rows, half of the columns each) read one out
// while the next tile's products run and store it with lanes along the columns.  Every wait is bounded.
#include "tcgen05.cuh"

#define HT_BM 128
#define HT_BK 64
#define HT_EPI_WARPS 8
#define HT_THREADS (64 + HT_EPI_WARPS * 32)

static __device__ int g_tc_status = 0;

template <int BN> struct HtShape { static constexpr int STAGES = BN <= 128 ? 5 : 4; };
template <int BN>
struct __align__(1024) HtSmem {
  __nv_bfloat16 a[HtShape<BN>::STAGES][HT_BM * HT_BK];
  __nv_bfloat16 b[HtShape<BN>::STAGES][BN * HT_BK];
  unsigned char stage[HT_EPI_WARPS][4096];
  uint64_t full[HtShape<BN>::STAGES], empty[HtShape<BN>::STAGES];
  uint64_t acc_full[2], acc_empty[2];
  uint32_t tmem_base;
  int abort_flag;
};

template <int BN>
__global__ void __launch_bounds__(HT_THREADS, 1)
head_linear_tc_kernel(const __grid_constant__ CUtensorMap map_x, const __grid_constant__ CUtensorMap map_w, __nv_bfloat16* __restrict__ out,
                      long ldo, long ldo_h, int M, int H, int N, int K, const __nv_bfloat16* __restrict__ gate, long ldg) {
  extern __shared__ unsigned char smem_raw[];
  constexpr int STAGES = HtShape<BN>::STAGES;
  constexpr uint32_t BUF = BN <= 64 ? 64 : BN <= 128 ? 128 : 256;         // columns between the two accumulators
  constexpr uint32_t STAGE_BYTES = (HT_BM + BN) * HT_BK * sizeof(__nv_bfloat16);
  pdl_launch_dependents();
  HtSmem<BN>& sm = *reinterpret_cast<HtSmem<BN>*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int num_kb = (K + HT_BK - 1) / HT_BK;
  const int n_blocks = (N + BN - 1) / BN;
  const int n_tiles = n_blocks * H * ((M + HT_BM - 1) / HT_BM);
  volatile int* abort_flag = &sm.abort_flag;
  if (threadIdx.x == 0) {
    tma_prefetch_map(&map_x);
    tma_prefetch_map(&map_w);
    for (int s = 0; s < STAGES; ++s) { mbar_init(&sm.full[s], 1); mbar_init(&sm.empty[s], 1); }
    for (int s = 0; s < 2; ++s) { mbar_init(&sm.acc_full[s], 1); mbar_init(&sm.acc_empty[s], HT_EPI_WARPS); }
    sm.abort_flag = 0;
    mbar_init_fence();
  }
  if (warp == 1) tc_alloc(&sm.tmem_base, 2 * BUF);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = sm.tmem_base;
  pdl_wait();
  auto tile_at = [&](int tile, int& m0, int& h, int& n0) {                // a token tile's heads one after the other
    n0 = (tile % n_blocks) * BN;
    h = (tile / n_blocks) % H;
    m0 = (tile / n_blocks / H) * HT_BM;
  };
  if (warp == 0) {
    if (lane == 0) {
      uint32_t kc = 0;
      bool ok = true;
      for (int tile = blockIdx.x; ok && tile < n_tiles; tile += gridDim.x) {
        int m0, h, n0;
        tile_at(tile, m0, h, n0);
        for (int kb = 0; kb < num_kb; ++kb, ++kc) {
          const uint32_t s = kc % STAGES, round = kc / STAGES;
          if (round > 0 && !mbar_wait(&sm.empty[s], (round - 1) & 1, abort_flag, 61, &g_tc_status)) { ok = false; break; }
          mbar_expect_tx(&sm.full[s], STAGE_BYTES);
          tma_load_3d(sm.a[s], &map_x, &sm.full[s], kb * HT_BK, h, m0);
          tma_load_3d(sm.b[s], &map_w, &sm.full[s], kb * HT_BK, n0, h);
        }
      }
      if (!ok) {
        // giving up: let the copies that are still in flight land before the CTA leaves (bounded)
        for (uint32_t i = kc > (uint32_t)STAGES ? kc - STAGES : 0; i < kc; ++i)
          for (uint32_t spin = 0; spin < TC_WAIT_LIMIT; ++spin)
            if (mbar_try_wait(&sm.full[i % STAGES], (i / STAGES) & 1)) break;
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc = make_idesc(HT_BM, BN);
      uint32_t kc = 0;
      bool ok = true;
      int it = 0;
      for (int tile = blockIdx.x; ok && tile < n_tiles; tile += gridDim.x, ++it) {
        const int buf = it & 1;
        if (it >= 2 && !mbar_wait(&sm.acc_empty[buf], ((it >> 1) - 1) & 1, abort_flag, 64, &g_tc_status)) { ok = false; break; }
        tc_fence_after();
        for (int kb = 0; kb < num_kb; ++kb, ++kc) {
          const uint32_t s = kc % STAGES;
          if (!mbar_wait(&sm.full[s], (kc / STAGES) & 1, abort_flag, 62, &g_tc_status)) { ok = false; break; }
          tc_fence_after();
          const uint64_t da = make_smem_desc(smem_u32(sm.a[s])), db = make_smem_desc(smem_u32(sm.b[s]));
#pragma unroll
          for (int k = 0; k < HT_BK / 16; ++k) tc_mma_bf16(tmem + buf * BUF, da + 2 * k, db + 2 * k, idesc, (kb | k) != 0);
          tc_commit(&sm.empty[s]);
        }
        if (ok) tc_commit(&sm.acc_full[buf]);
      }
    }
  } else {
    const int quarter = warp & 3, half = (warp - 2) >> 2;
    int it = 0;
    for (int tile = blockIdx.x; tile < n_tiles; tile += gridDim.x, ++it) {
      const int buf = it & 1;
      int m0, h, n0;
      tile_at(tile, m0, h, n0);
      const int row = m0 + quarter * 32 + lane;
      float f = 1.f;
      if (gate != nullptr && row < M) f = 1.f / (1.f + expf(-__bfloat162float(gate[(size_t)row * ldg + h])));
      if (!__all_sync(0xffffffffu, mbar_wait(&sm.acc_full[buf], (it >> 1) & 1, abort_flag, 63, &g_tc_status))) break;
      tc_fence_after();
#pragma unroll 1
      for (int c0 = half * (BN / 2); c0 < (half + 1) * (BN / 2); c0 += 32) {
        uint32_t v[32], p[16];
        tc_ld_32x32b_x32(tmem + ((uint32_t)(quarter * 32) << 16) + buf * BUF + c0, v);
        tc_wait_ld();
        if (c0 + 32 == (half + 1) * (BN / 2)) {
          tc_fence_before();
          __syncwarp();
          if (lane == 0) mbar_arrive(&sm.acc_empty[buf]);
        }
#pragma unroll
        for (int j = 0; j < 32; j += 2) {
          __nv_bfloat162 b2 = __floats2bfloat162_rn(__uint_as_float(v[j]) * f, __uint_as_float(v[j + 1]) * f);
          p[j >> 1] = *reinterpret_cast<uint32_t*>(&b2);
        }
        const int r_first = m0 + quarter * 32;
        pr_store_block<32>(sm.stage[warp - 2], p, out + (size_t)r_first * ldo + (size_t)h * ldo_h + n0 + c0, (size_t)ldo, M - r_first,
                           N - (n0 + c0), lane);
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tc_dealloc(tmem, 2 * BUF);
  }
}

extern "C" int qe_head_linear_tc_status() {
  int v = 0;
  cudaMemcpyFromSymbol(&v, g_tc_status, sizeof(int));
  return v;
}
extern "C" void qe_head_linear_tc_clear_status() {
  int v = 0;
  cudaMemcpyToSymbol(g_tc_status, &v, sizeof(int));
}

template <int BN>
static int launch_head_linear_tc(const void* x, long ldx, long ldx_h, const void* w, void* out, long ldo, long ldo_h, int M, int H, int N,
                                 int K, const void* gate, long ldg, cudaStream_t stream) {
  CUtensorMap map_x, map_w;
  {
    const uint64_t dims[3] = {(uint64_t)K, (uint64_t)H, (uint64_t)M};
    const uint64_t strides[2] = {(uint64_t)ldx_h * 2, (uint64_t)ldx * 2};
    const uint32_t box[3] = {HT_BK, 1, HT_BM};
    if (!qe_tensor_map_bf16(x, 3, dims, strides, box, &map_x)) return 1;
  }
  {
    const uint64_t dims[3] = {(uint64_t)K, (uint64_t)N, (uint64_t)H};
    const uint64_t strides[2] = {(uint64_t)K * 2, (uint64_t)K * 2 * (uint64_t)N};
    const uint32_t box[3] = {HT_BK, BN, 1};
    if (!qe_tensor_map_bf16(w, 3, dims, strides, box, &map_w)) return 1;
  }
  const size_t smem = sizeof(HtSmem<BN>) + 1024;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(head_linear_tc_kernel<BN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) QE_REFUSE("head_linear_tc: shared memory %zu: %s", smem, cudaGetErrorString(e));
    configured = true;
  }
  static int sms = 0;
  if (sms == 0) {
    int dev = 0, v = 148;
    if (cudaGetDevice(&dev) == cudaSuccess) cudaDeviceGetAttribute(&v, cudaDevAttrMultiProcessorCount, dev);
    sms = v > 0 ? v : 148;
  }
  const long tiles = (long)((N + BN - 1) / BN) * H * ((M + HT_BM - 1) / HT_BM);
  if (tiles > 0x7fffffffL) QE_REFUSE("head_linear_tc: %ld tiles", tiles);
  qe_launch(head_linear_tc_kernel<BN>, dim3((unsigned)(tiles < sms ? tiles : sms)), dim3(HT_THREADS), smem, stream, map_x, map_w,
            (__nv_bfloat16*)out, ldo, ldo_h, M, H, N, K, (const __nv_bfloat16*)gate, ldg);
  QE_CHECK_LAUNCH("head_linear_tc");
  return 0;
}

// Arguments as qe_head_linear (bfloat16).  K a multiple of 8, strides of x and out multiples of 8 elements, all on 16-byte boundaries.
extern "C" int qe_head_linear_tc(const void* x, long ldx, long ldx_h, const void* w, void* out, long ldo, long ldo_h, int M, int H,
                                 int N, int K, const void* gate, long ldg, cudaStream_t stream) {
  if (M <= 0 || H <= 0 || N <= 0) return 0;
  if (K < 8 || K % 8 || ldx % 8 || ldx_h % 8 || ldo % 8 || ldo_h % 8) QE_REFUSE("head_linear_tc: K = %d or strides that are no multiples of 8", K);
  if (((uintptr_t)x | (uintptr_t)w | (uintptr_t)out) & 15) QE_REFUSE("head_linear_tc: operands must be 16-byte aligned");
#define HT_GO(BN) return launch_head_linear_tc<BN>(x, ldx, ldx_h, w, out, ldo, ldo_h, M, H, N, K, gate, ldg, stream)
  if (N <= 64) HT_GO(64);
  if (N <= 128) HT_GO(128);
  if (N <= 192) HT_GO(192);
  HT_GO(256);
#undef HT_GO
}
