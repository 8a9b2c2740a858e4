// PTX wrappers of the fifth-generation tensor-core path (sm_100a): mbarriers with bounded waits, TMA
// tile loads, tcgen05 matrix instructions, tensor-memory loads and stores, operand descriptors; and
// the host-side cache of TMA tensor maps.  Shared by the kernels that use tcgen05.
#pragma once
#include "common.cuh"
#include <cuda.h>

#define TC_WAIT_LIMIT (1u << 22)     // polls of a barrier before giving up (each poll may itself block for a while)

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }

// ---- mbarriers ------------------------------------------------------------------------------------------
__device__ __forceinline__ void mbar_init(uint64_t* bar, uint32_t count) {
  asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;\n" :: "r"(smem_u32(bar)), "r"(count));
}
__device__ __forceinline__ void mbar_init_fence() { asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory"); }
__device__ __forceinline__ void mbar_arrive(uint64_t* bar) {
  asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];\n" :: "r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ void mbar_expect_tx(uint64_t* bar, uint32_t bytes) {
  asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;\n" :: "r"(smem_u32(bar)), "r"(bytes) : "memory");
}
__device__ __forceinline__ bool mbar_try_wait(uint64_t* bar, uint32_t parity) {
  uint32_t ok;
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\t"
      "selp.b32 %0, 1, 0, p;\n\t}\n"
      : "=r"(ok) : "r"(smem_u32(bar)), "r"(parity) : "memory");
  return ok != 0;
}
// Bounded wait: false if the barrier did not flip within the limit or the CTA is aborting.  A wait
// that runs out raises the CTA's abort flag and records `code` in `*status` (if nothing is there yet).
__device__ __forceinline__ bool mbar_wait(uint64_t* bar, uint32_t parity, volatile int* abort_flag, int code, int* status,
                                          uint32_t limit = TC_WAIT_LIMIT) {
  for (uint32_t i = 0; i < limit; ++i) {
    if (mbar_try_wait(bar, parity)) return true;
    if ((i & 63) == 63 && *abort_flag) return false;
  }
  *abort_flag = 1;
  atomicCAS(status, 0, code);
  return false;
}

// ---- TMA tile loads (no multicast: every CTA fetches its own tiles) -------------------------------------------
__device__ __forceinline__ void tma_load_2d(void* dst, const CUtensorMap* map, uint64_t* bar, int c0, int c1) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4}], [%2];\n"
      :: "r"(smem_u32(dst)), "l"(map), "r"(smem_u32(bar)), "r"(c0), "r"(c1) : "memory");
}
__device__ __forceinline__ void tma_load_3d(void* dst, const CUtensorMap* map, uint64_t* bar, int c0, int c1, int c2) {
  asm volatile(
      "cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];\n"
      :: "r"(smem_u32(dst)), "l"(map), "r"(smem_u32(bar)), "r"(c0), "r"(c1), "r"(c2) : "memory");
}
__device__ __forceinline__ void tma_load_5d(void* dst, const CUtensorMap* map, uint64_t* bar, int c0, int c1, int c2,
                                            int c3, int c4) {
  asm volatile(
      "cp.async.bulk.tensor.5d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5, %6, %7}], [%2];\n"
      :: "r"(smem_u32(dst)), "l"(map), "r"(smem_u32(bar)), "r"(c0), "r"(c1), "r"(c2), "r"(c3), "r"(c4) : "memory");
}

// bring a tensor map (a kernel parameter) into the TMA unit's cache before the first load that uses it
__device__ __forceinline__ void tma_prefetch_map(const CUtensorMap* map) {
  asm volatile("prefetch.tensormap [%0];\n" :: "l"(map) : "memory");
}

// ---- tcgen05 ---------------------------------------------------------------------------------------------
__device__ __forceinline__ void tc_fence_before() { asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory"); }
__device__ __forceinline__ void tc_fence_after() { asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory"); }
__device__ __forceinline__ void tc_commit(uint64_t* bar) {
  asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];\n" :: "r"(smem_u32(bar)) : "memory");
}
// D[tmem] (+)= A[smem] · B[smem]
__device__ __forceinline__ void tc_mma_bf16(uint32_t d_tmem, uint64_t a_desc, uint64_t b_desc, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}\n"
      :: "r"(d_tmem), "l"(a_desc), "l"(b_desc), "r"(idesc), "r"(accumulate) : "memory");
}
// D[tmem] (+)= A[tmem] · B[smem]: A's rows are the lanes, two bfloat16 of consecutive k per 32-bit column
__device__ __forceinline__ void tc_mma_bf16_ts(uint32_t d_tmem, uint32_t a_tmem, uint64_t b_desc, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}\n"
      :: "r"(d_tmem), "r"(a_tmem), "l"(b_desc), "r"(idesc), "r"(accumulate) : "memory");
}
// lane i of the warp gets columns taddr.col .. +31 of tensor-memory lane taddr.lane + i
__device__ __forceinline__ void tc_ld_32x32b_x32(uint32_t taddr, uint32_t (&r)[32]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 "
      "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, "
      "%16, %17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31}, [%32];\n"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]),
        "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]),
        "=r"(r[16]), "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]), "=r"(r[23]),
        "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
      : "r"(taddr) : "memory");
}
__device__ __forceinline__ void tc_st_32x32b_x32(uint32_t taddr, const uint32_t (&r)[32]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%32], "
      "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, "
      "%16, %17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31};\n"
      :: "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]),
         "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]),
         "r"(r[16]), "r"(r[17]), "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]),
         "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31]),
         "r"(taddr) : "memory");
}
__device__ __forceinline__ void tc_wait_ld() { asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory"); }
__device__ __forceinline__ void tc_wait_st() { asm volatile("tcgen05.wait::st.sync.aligned;\n" ::: "memory"); }

// One warp allocates `cols` columns (a power of two, 32..512) of tensor memory and writes their base
// address to shared memory; the same warp frees them.
__device__ __forceinline__ void tc_alloc(uint32_t* result_in_smem, uint32_t cols) {
  asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n"
               :: "r"(smem_u32(result_in_smem)), "r"(cols) : "memory");
  asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::: "memory");
}
__device__ __forceinline__ void tc_dealloc(uint32_t tmem, uint32_t cols) {
  asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" :: "r"(tmem), "r"(cols) : "memory");
}

// ---- CTA pairs (cta_group::2): two CTAs of a cluster, on neighbouring SMs, work on one tile -------------------
// A shared-memory address of the odd CTA of a pair differs from the same offset in the even CTA by
// this bit; with it cleared, an address names the even ("leading") CTA's copy.
#define TC_PEER_BIT_MASK 0xFEFFFFFFu

// arrive on a barrier that may lie in the other CTA of the cluster (bar_addr: a shared::cluster address)
__device__ __forceinline__ void mbar_arrive_cluster(uint32_t bar_addr) {
  asm volatile("mbarrier.arrive.release.cluster.shared::cluster.b64 _, [%0];\n" :: "r"(bar_addr) : "memory");
}
// TMA tile load into this CTA's shared memory whose bytes are counted on a barrier of either CTA of the pair
__device__ __forceinline__ void tma_load_2d_pair(void* dst, const CUtensorMap* map, uint32_t bar_addr, int c0, int c1) {
  asm volatile(
      "cp.async.bulk.tensor.2d.cta_group::2.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4}], [%2];\n"
      :: "r"(smem_u32(dst)), "l"(map), "r"(bar_addr), "r"(c0), "r"(c1) : "memory");
}
// both CTAs of the pair execute these with the same arguments
__device__ __forceinline__ void tc_alloc_pair(uint32_t* result_in_smem, uint32_t cols) {
  asm volatile("tcgen05.alloc.cta_group::2.sync.aligned.shared::cta.b32 [%0], %1;\n"
               :: "r"(smem_u32(result_in_smem)), "r"(cols) : "memory");
  asm volatile("tcgen05.relinquish_alloc_permit.cta_group::2.sync.aligned;\n" ::: "memory");
}
__device__ __forceinline__ void tc_dealloc_pair(uint32_t tmem, uint32_t cols) {
  asm volatile("tcgen05.dealloc.cta_group::2.sync.aligned.b32 %0, %1;\n" :: "r"(tmem), "r"(cols) : "memory");
}
// issued by one thread of the leading CTA: D[tmem of both] (+)= A[256 rows: 128 of each CTA] · B[N: N/2 of each CTA]
__device__ __forceinline__ void tc_mma_bf16_pair(uint32_t d_tmem, uint64_t a_desc, uint64_t b_desc, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::2.kind::f16 [%0], %1, %2, %3, p;\n\t}\n"
      :: "r"(d_tmem), "l"(a_desc), "l"(b_desc), "r"(idesc), "r"(accumulate) : "memory");
}
// arrives on the barrier at this offset in every CTA of `cta_mask` when the pair's earlier MMAs have retired
__device__ __forceinline__ void tc_commit_pair(uint64_t* bar, uint16_t cta_mask) {
  asm volatile("tcgen05.commit.cta_group::2.mbarrier::arrive::one.shared::cluster.multicast::cluster.b64 [%0], %1;\n"
               :: "r"(smem_u32(bar)), "h"(cta_mask) : "memory");
}

// Shared-memory matrix descriptor of a K-major tile with 128-byte swizzle (rows of 64 bfloat16 = 128
// bytes, groups of 8 rows = 1024 bytes): start address, leading offset 1, stride offset 1024 bytes
// (both in 16-byte units), descriptor version 1, layout type 2 (128-byte swizzle).
__device__ __forceinline__ uint64_t make_smem_desc(uint32_t addr) {
  return (uint64_t)((addr >> 4) & 0x3fff) | (1ull << 16) | ((uint64_t)(1024 >> 4) << 32) | (1ull << 46) | (2ull << 61);
}
// The same for an MN-major tile with 128-byte swizzle: rows are k, a row holds 64 consecutive
// elements of the M or N dimension (128 bytes); groups of 8 rows (1024 bytes) follow one another at
// `k_group_bytes`, the next 64 elements of M or N lie `mn_block_bytes` further.
__device__ __forceinline__ uint64_t make_smem_desc_mn(uint32_t addr, uint32_t mn_block_bytes, uint32_t k_group_bytes) {
  return (uint64_t)((addr >> 4) & 0x3fff) | ((uint64_t)((mn_block_bytes >> 4) & 0x3fff) << 16) |
         ((uint64_t)((k_group_bytes >> 4) & 0x3fff) << 32) | (1ull << 46) | (2ull << 61);
}
// Instruction descriptor: D float32, A and B bfloat16, N / 8 at bit 17, M / 16 at bit 24; bit 16 set
// when B is MN-major (else both operands are K-major).
__host__ __device__ constexpr uint32_t make_idesc(int M, int N, bool b_mn_major = false) {
  return (1u << 4) | (1u << 7) | (1u << 10) | (b_mn_major ? (1u << 16) : 0u) | ((uint32_t)(N >> 3) << 17) |
         ((uint32_t)(M >> 4) << 24);
}

// 32 rows x COLS bfloat16 columns of the output, from the warp whose lane l holds row l (as the accumulator leaves
// tensor memory: packed[i] = columns 2 i, 2 i + 1 of the lane's row), to memory with lanes along the columns: through
// 4 KB of shared memory of the warp's own (16-byte chunks XORed with the row's low bits), then 128 or 64 bytes of a
// row per 8 or 4 lanes.  Stored with lanes along the rows, every instruction touched 32 rows with 16 bytes each, and a
// tile's epilogue took 3.5-5.8 us (measured with the timeline build), as long as its products.
// dst: row 0, column 0 of the 32 x COLS block; ld: elements per row of the output; rows, cols: how many of them exist.
template <int COLS>
__device__ __forceinline__ void pr_store_block(unsigned char* wst, const uint32_t (&packed)[COLS / 2], __nv_bfloat16* dst, size_t ld,
                                               int rows, int cols, int lane) {
  constexpr int CH = COLS / 8, RB = COLS * 2, RPI = 32 / CH;     // chunks per row, bytes per row, rows per instruction
#pragma unroll
  for (int j = 0; j < CH; ++j)
    *reinterpret_cast<uint4*>(wst + lane * RB + ((j ^ (lane & (CH - 1))) << 4)) =
        make_uint4(packed[4 * j], packed[4 * j + 1], packed[4 * j + 2], packed[4 * j + 3]);
  __syncwarp();
  const int cj = lane % CH;
#pragma unroll
  for (int i = 0; i < CH; ++i) {
    const int rr = i * RPI + lane / CH;
    const uint4 v = *reinterpret_cast<const uint4*>(wst + rr * RB + ((cj ^ (rr & (CH - 1))) << 4));
    if (rr < rows) {
      __nv_bfloat16* d = dst + (size_t)rr * ld + cj * 8;
      if (cj * 8 + 8 <= cols) {
        *reinterpret_cast<uint4*>(d) = v;
      } else {
        const __nv_bfloat16* e = reinterpret_cast<const __nv_bfloat16*>(&v);
        for (int k = 0; k < 8; ++k)
          if (cj * 8 + k < cols) d[k] = e[k];
      }
    }
  }
  __syncwarp();
}

// ---- host side: TMA tensor maps, cached by what they describe ---------------------------------------------------
// A bfloat16 tensor of `rank` dimensions (innermost first): extents, strides in bytes of dimensions
// 1.. (the innermost is dense), box; 128-byte swizzle, zero fill outside.  False (with the error text
// set) if the driver refuses.
bool qe_tensor_map_bf16(const void* ptr, int rank, const uint64_t* dims, const uint64_t* strides_bytes,
                        const uint32_t* box, CUtensorMap* out);
