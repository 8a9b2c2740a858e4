// Attention of prompt portions over a latent cache in bfloat16 on tcgen05: one key per token of D channels that all query
// heads share and whose first channels are also the value (latent_attention.cu), D a multiple of 16 up to 256.
//
// The queries of a token's heads lie side by side, so q [T, H D] is a matrix of T H rows of D channels and a tile is 128
// consecutive ones of them, whatever H is (as many whole tokens as fit; the rows behind them are computed and not stored).
// One CTA serves a tile; its keys come in steps of 64 through a ring of slots by TMA out of the pages (a box per page and 64
// channels; the box of a page that is not held lies outside the tensor and is filled with zeros).  A slot is the K-major
// operand of S = Q K^T and, read with rows as k, the MN-major operand of O += P V: a key is fetched once for both.  S (four
// buffers of 64 columns), P (bfloat16, in the place of its S, the A operand from tensor memory) and O (up to 256 columns)
// live in tensor memory.
//
// 6 warps: warp 0 issues the loads, one thread of warp 1 the MMAs, warps 2 to 5 (a thread per row) mask, exponentiate and
// keep the row's maximum and sum in float32; O is rescaled only when a row's maximum has grown by more than 2^8.  A head's
// sink joins its row's denominator at the end.  Every wait is bounded (status word).  Keys of a held page past the
// request's length are read as they are and masked, so pages must hold finite values.
//
// Work items are those of the flash kernel (attention_flash.cuh), one per tile, longest first.
#include "tcgen05.cuh"
#include <math.h>

#define LT_ROWS 128
#define LT_BN 64
#define LT_S_BUFS 4
#define LT_THREADS 192
#define LT_MAX_SLOTS 8
#define LT_ITEM_INTS 12
#define LT_LOG2E 1.4426950408889634f
#define LT_LAZY 8.f                       // how far (in powers of two) a row's maximum may grow before O is rescaled

static __device__ int g_lt_status = 0;

struct LtArgs {
  const int* items; const int* block_tables; int max_blocks, num_pages;
  __nv_bfloat16* out;
  const float* sinks;
  float scale_log2;
  int window, H, D, v_pad, page_size, col_blocks, slots;
};

struct LtBars {
  uint64_t q_full, k_full[LT_MAX_SLOTS], k_empty[LT_MAX_SLOTS];
  uint64_t s_full[LT_S_BUFS], p_full[LT_S_BUFS], pv_done[LT_S_BUFS];
  uint32_t tmem_base;
  int abort_flag;
};

__device__ __forceinline__ float lt_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
  return y;
}

__global__ void __launch_bounds__(LT_THREADS, 1)
latent_attention_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_kv, LtArgs A) {
  extern __shared__ unsigned char smem_raw[];
  __shared__ LtBars bars;
  pdl_launch_dependents();
  unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int CB = A.col_blocks, SLOTS = A.slots;
  unsigned char* sq = smem;                                       // [CB][128 rows][128 bytes]
  unsigned char* sk = smem + (size_t)CB * LT_ROWS * 128;          // [slots][CB][64 keys][128 bytes]
  const uint32_t slot_bytes = (uint32_t)CB * LT_BN * 128u;
  volatile int* abort_flag = &bars.abort_flag;

  // the work lists come from the host's copy, not from a kernel
  const int* it = A.items + (size_t)blockIdx.x * LT_ITEM_INTS;
  const int req = it[0], q0 = it[1], row0 = it[7], q_len = it[8], ctx = it[9];
  const int H = A.H;
  const int ntok = min(LT_ROWS / H, q_len - q0);
  const int nrows = ntok * H;
  const int first_pos = ctx + q0;
  const int kv_end = first_pos + ntok;
  const int kv_begin = A.window > 0 ? max(0, first_pos - A.window + 1) : 0;
  const int kt0 = kv_begin / LT_BN * LT_BN;
  const int n_steps = (kv_end - kt0 + LT_BN - 1) / LT_BN;         // at least one: a token sees itself

  if (threadIdx.x == 0) {
    tma_prefetch_map(&map_q);
    tma_prefetch_map(&map_kv);
    mbar_init(&bars.q_full, 1);
    for (int s = 0; s < SLOTS; ++s) { mbar_init(&bars.k_full[s], 1); mbar_init(&bars.k_empty[s], 1); }
    for (int s = 0; s < LT_S_BUFS; ++s) { mbar_init(&bars.s_full[s], 1); mbar_init(&bars.p_full[s], 4); mbar_init(&bars.pv_done[s], 1); }
    bars.abort_flag = 0;
    mbar_init_fence();
  }
  if (warp == 1) tc_alloc(&bars.tmem_base, 512);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = bars.tmem_base;                           // S buffers at 0, 64, 128, 192; O from 256 on
  pdl_wait();

  if (warp == 0) {
    // the whole warp issues the loads, a lane per box of a step (a page and 64 channels)
    if (lane == 0) mbar_expect_tx(&bars.q_full, (uint32_t)CB * LT_ROWS * 128u);
    __syncwarp();
    if (lane < CB) tma_load_2d(sq + (size_t)lane * LT_ROWS * 128, &map_q, &bars.q_full, lane * 64, (row0 + q0) * H);
    const int* table = A.block_tables + (size_t)req * A.max_blocks;
    const int box_rows = min(A.page_size, LT_BN);                 // (a power of two, at least 8: at most 8 boxes of 4 blocks a step)
    const int page_shift = __ffs(A.page_size) - 1;
    const int b = lane / CB, cb = lane - b * CB;
    const bool mine = b < LT_BN / box_rows;
    auto page_of = [&](int j) {                                   // the page of this lane's box of step j
      const int key = kt0 + j * LT_BN + b * box_rows, blk = key >> page_shift;
      int page = (mine && j < n_steps && key < kv_end && key + box_rows > kv_begin && blk < A.max_blocks) ? __ldg(table + blk) : -1;
      return page < 0 ? A.num_pages : page;                       // outside the tensor: zeros
    };
    bool ok = true;
    int j = 0, page = page_of(0);
    for (; j < n_steps; ++j) {
      const int s = j % SLOTS, round = j / SLOTS;
      const int next_page = page_of(j + 1);
      if (round > 0) ok = __all_sync(0xffffffffu, mbar_wait(&bars.k_empty[s], (round - 1) & 1, abort_flag, 51, &g_lt_status));
      if (!ok) break;
      if (lane == 0) mbar_expect_tx(&bars.k_full[s], slot_bytes);
      __syncwarp();
      if (mine)
        tma_load_3d(sk + (size_t)s * slot_bytes + ((size_t)cb * LT_BN + (size_t)b * box_rows) * 128, &map_kv, &bars.k_full[s],
                    cb * 64, (kt0 + j * LT_BN + b * box_rows) & (A.page_size - 1), page);
      page = next_page;
    }
    if (!ok && lane == 0) {
      // giving up: let the copies that are still in flight land before the CTA leaves (bounded)
      for (uint32_t spin = 0; spin < TC_WAIT_LIMIT; ++spin) if (mbar_try_wait(&bars.q_full, 0)) break;
      for (int i = j > SLOTS ? j - SLOTS : 0; i < j; ++i)
        for (uint32_t spin = 0; spin < TC_WAIT_LIMIT; ++spin) if (mbar_try_wait(&bars.k_full[i % SLOTS], (i / SLOTS) & 1)) break;
    }
    __syncwarp();
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc_s = make_idesc(LT_ROWS, LT_BN);
      const uint32_t idesc_o = make_idesc(LT_ROWS, A.v_pad, true);
      const int nks = A.D >> 4;
      const uint32_t q_addr = smem_u32(sq), k_addr = smem_u32(sk);
      auto issue_s = [&](int j) -> bool {
        const int s = j % SLOTS, b = j % LT_S_BUFS;
        if (!mbar_wait(&bars.k_full[s], (j / SLOTS) & 1, abort_flag, 52, &g_lt_status)) return false;
        // the buffer's last P has been read by its product
        if (j >= LT_S_BUFS && !mbar_wait(&bars.pv_done[b], (j / LT_S_BUFS - 1) & 1, abort_flag, 53, &g_lt_status)) return false;
        tc_fence_after();
        for (int ks = 0; ks < nks; ++ks) {
          const uint64_t da = make_smem_desc(q_addr + (uint32_t)(ks >> 2) * (LT_ROWS * 128u)) + 2 * (ks & 3);
          const uint64_t db = make_smem_desc(k_addr + (uint32_t)s * slot_bytes + (uint32_t)(ks >> 2) * (LT_BN * 128u)) + 2 * (ks & 3);
          tc_mma_bf16(tmem + b * LT_BN, da, db, idesc_s, ks != 0);
        }
        tc_commit(&bars.s_full[b]);
        return true;
      };
      bool ok = mbar_wait(&bars.q_full, 0, abort_flag, 54, &g_lt_status);
      int ahead = 0;
      // scores run up to two steps ahead of the products with the values
      for (int j = 0; ok && j < n_steps; ++j) {
        while (ok && ahead < n_steps && ahead <= j + 2) { ok = issue_s(ahead); ++ahead; }
        if (!ok) break;
        const int s = j % SLOTS, b = j % LT_S_BUFS;
        if (!mbar_wait(&bars.p_full[b], (j / LT_S_BUFS) & 1, abort_flag, 55, &g_lt_status)) { ok = false; break; }
        tc_fence_after();
        const uint64_t dv = make_smem_desc_mn(k_addr + (uint32_t)s * slot_bytes, LT_BN * 128, 1024);
#pragma unroll
        for (int ks = 0; ks < LT_BN / 16; ++ks)
          tc_mma_bf16_ts(tmem + 256, tmem + b * LT_BN + ks * 8, dv + ks * (2048 >> 4), idesc_o, (j | ks) != 0);
        tc_commit(&bars.k_empty[s]);
        tc_commit(&bars.pv_done[b]);
      }
    }
  } else {
    // ---- a thread per row ------------------------------------------------------------------------------------------------
    const int quarter = warp & 3;
    const uint32_t lane_base = tmem + ((uint32_t)(quarter * 32) << 16);
    const int r = quarter * 32 + lane;
    const int pos = first_pos + min(r, nrows - 1) / H;
    const int pos_first = first_pos + min(quarter * 32, nrows - 1) / H;           // of the warp's rows
    const int pos_last = first_pos + min(quarter * 32 + 31, nrows - 1) / H;
    const int low = A.window > 0 ? pos - A.window : -1;                            // keys above it are seen
    float m_used = -INFINITY, l_run = 0.f;
    bool ok = true;
    for (int j = 0; j < n_steps; ++j) {
      const int b = j % LT_S_BUFS;
      const int kt = kt0 + j * LT_BN;
      ok = __all_sync(0xffffffffu, mbar_wait(&bars.s_full[b], (j / LT_S_BUFS) & 1, abort_flag, 56, &g_lt_status));
      if (!ok) break;
      tc_fence_after();
      uint32_t s[2][32];
      tc_ld_32x32b_x32(lane_base + b * LT_BN, s[0]);
      tc_ld_32x32b_x32(lane_base + b * LT_BN + 32, s[1]);
      tc_wait_ld();
      float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
      const bool all = kt + LT_BN - 1 <= pos_first && (A.window <= 0 || kt > pos_last - A.window);
      if (all) {
#pragma unroll
        for (int q = 0; q < 2; ++q)
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            const float v = __uint_as_float(s[q][i]) * A.scale_log2;
            s[q][i] = __float_as_uint(v);
            mx[i & 3] = fmaxf(mx[i & 3], v);
          }
      } else {
#pragma unroll
        for (int q = 0; q < 2; ++q)
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            const int key = kt + q * 32 + i;
            const float v = key <= pos && key > low ? __uint_as_float(s[q][i]) * A.scale_log2 : -INFINITY;
            s[q][i] = __float_as_uint(v);
            mx[i & 3] = fmaxf(mx[i & 3], v);
          }
      }
      const float m_tile = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3]));
      float alpha = 1.f;
      const bool grow = m_tile > m_used + LT_LAZY || (m_used == -INFINITY && m_tile > -INFINITY);
      if (grow) { alpha = lt_exp2(m_used - m_tile); m_used = m_tile; l_run *= alpha; }
      if (j > 0 && __any_sync(0xffffffffu, grow)) {
        // O is rescaled once its last product has retired
        ok = __all_sync(0xffffffffu, mbar_wait(&bars.pv_done[(j - 1) % LT_S_BUFS], ((j - 1) / LT_S_BUFS) & 1, abort_flag, 57, &g_lt_status));
        if (!ok) break;
        tc_fence_after();
        for (int c = 0; c < A.v_pad; c += 32) {
          uint32_t o[32];
          tc_ld_32x32b_x32(lane_base + 256 + c, o);
          tc_wait_ld();
#pragma unroll
          for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
          tc_st_32x32b_x32(lane_base + 256 + c, o);
        }
      }
      const float base = m_used == -INFINITY ? 0.f : m_used;
      float sum[4] = {0.f, 0.f, 0.f, 0.f};
      uint32_t p[32];
#pragma unroll
      for (int q = 0; q < 2; ++q)
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          const float e0 = lt_exp2(__uint_as_float(s[q][i]) - base), e1 = lt_exp2(__uint_as_float(s[q][i + 1]) - base);
          sum[i & 2] += e0;
          sum[(i & 2) + 1] += e1;
          __nv_bfloat162 h2 = __floats2bfloat162_rn(e0, e1);
          p[q * 16 + (i >> 1)] = *reinterpret_cast<uint32_t*>(&h2);
        }
      l_run += (sum[0] + sum[1]) + (sum[2] + sum[3]);
      tc_st_32x32b_x32(lane_base + b * LT_BN, p);
      tc_wait_st();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars.p_full[b]);
    }
    if (ok) ok = __all_sync(0xffffffffu, mbar_wait(&bars.pv_done[(n_steps - 1) % LT_S_BUFS], ((n_steps - 1) / LT_S_BUFS) & 1, abort_flag, 58, &g_lt_status));
    if (ok) {
      tc_fence_after();
      float l = l_run;
      // the sink's share of the denominator: exp(sink), no key and no value
      if (A.sinks) l += lt_exp2(A.sinks[min(r, nrows - 1) % H] * LT_LOG2E - m_used);
      const float inv = l > 0.f ? 1.f / l : 0.f;
      __nv_bfloat16* dst = A.out + ((size_t)(row0 + q0) * H + r) * A.D;
      for (int c = 0; c < A.v_pad; c += 32) {
        uint32_t o[32];
        tc_ld_32x32b_x32(lane_base + 256 + c, o);
        tc_wait_ld();
        if (r < nrows) {
#pragma unroll
          for (int i = 0; i < 32; i += 8) {
            if (c + i < A.v_pad) {
              uint32_t w[4];
#pragma unroll
              for (int k = 0; k < 4; ++k) {
                __nv_bfloat162 h2 = __floats2bfloat162_rn(__uint_as_float(o[i + 2 * k]) * inv, __uint_as_float(o[i + 2 * k + 1]) * inv);
                w[k] = *reinterpret_cast<uint32_t*>(&h2);
              }
              *reinterpret_cast<uint4*>(dst + c + i) = make_uint4(w[0], w[1], w[2], w[3]);
            }
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
    tc_dealloc(tmem, 512);
  }
}

static int lt_smem_of(int D, int* col_blocks, int* slots) {
  const int cb = (D + 63) / 64;
  const int q = cb * LT_ROWS * 128, slot = cb * LT_BN * 128, limit = 224 * 1024;
  int n = (limit - q) / slot;
  n = n > LT_MAX_SLOTS ? LT_MAX_SLOTS : n;
  *col_blocks = cb;
  *slots = n;
  return q + n * slot + 1024;
}

extern "C" int qe_latent_attention_tc_status() {
  int v = 0;
  cudaMemcpyFromSymbol(&v, g_lt_status, sizeof(int));
  return v;
}
extern "C" void qe_latent_attention_tc_clear_status() {
  int v = 0;
  cudaMemcpyToSymbol(g_lt_status, &v, sizeof(int));
}

// q [T, H D] contiguous, pages [num_pages, page, D], out [T, H D] (the first v_dim channels of every head, rounded up to a
// multiple of 16, are written); items: tiles of 128 / H tokens.  Returns 0 when run, 1 when refused, 2 on a launch error.
extern "C" int qe_latent_attention_tc(const void* q, int T, const void* pages, int num_pages, const int* block_tables, int max_blocks,
                                      const int* items, int n_items, void* out, float scale, int window, int H, int D, int v_dim,
                                      int page_size, const float* sinks, cudaStream_t stream) {
  if (n_items <= 0) return 0;
  if (D < 16 || D > 256 || D % 16 || H < 1 || H > LT_ROWS) QE_REFUSE("latent_attention_tc: %d heads over cache rows of %d channels", H, D);
  if (v_dim < 1 || v_dim > D) QE_REFUSE("latent_attention_tc: values of %d channels", v_dim);
  if (page_size < 8 || (page_size & (page_size - 1))) QE_REFUSE("latent_attention_tc: pages of %d tokens", page_size);
  if (((uintptr_t)q | (uintptr_t)pages | (uintptr_t)out) & 15) QE_REFUSE("latent_attention_tc: operands must be 16-byte aligned");
  CUtensorMap map_q, map_kv;
  {
    const uint64_t dims[2] = {(uint64_t)D, (uint64_t)T * (uint64_t)H};
    const uint64_t strides[1] = {(uint64_t)D * 2};
    const uint32_t box[2] = {64, LT_ROWS};
    if (!qe_tensor_map_bf16(q, 2, dims, strides, box, &map_q)) return 1;
  }
  {
    const uint64_t dims[3] = {(uint64_t)D, (uint64_t)page_size, (uint64_t)num_pages};
    const uint64_t strides[2] = {(uint64_t)D * 2, (uint64_t)D * 2 * (uint64_t)page_size};
    const uint32_t box[3] = {64, (uint32_t)(page_size < LT_BN ? page_size : LT_BN), 1};
    if (!qe_tensor_map_bf16(pages, 3, dims, strides, box, &map_kv)) return 1;
  }
  int col_blocks = 0, slots = 0;
  const int smem = lt_smem_of(D, &col_blocks, &slots);
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(latent_attention_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 225 * 1024);
    if (e != cudaSuccess) QE_REFUSE("latent_attention_tc: shared memory: %s", cudaGetErrorString(e));
    configured = true;
  }
  const LtArgs A{items, block_tables, max_blocks, num_pages, (__nv_bfloat16*)out, sinks, scale * LT_LOG2E, window, H, D,
                 (v_dim + 15) / 16 * 16, page_size, col_blocks, slots};
  qe_launch(latent_attention_tc_kernel, dim3(n_items), dim3(LT_THREADS), (size_t)smem, stream, map_q, map_kv, A);
  QE_CHECK_LAUNCH("latent_attention_tc");
  return 0;
}
