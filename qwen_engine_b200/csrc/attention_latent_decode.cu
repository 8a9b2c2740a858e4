// Attention of decoded tokens over a latent cache in bfloat16: one key per token of D channels that all query heads
// share and whose first v_dim channels are also the value (see latent_attention.cu), D a multiple of 16 up to 256.
// The rows of a request (token x query head) ride the 16 rows of mma.sync.m16n8k16; every key is fetched once for
// 16 of them and serves both products out of the same shared memory.
//
// One CTA of 8 warps serves one work item (a request's rows, a range of its keys) and 16 of its rows.  The keys are
// dealt to the warps in groups of 16 that start at multiples of 16 (so a group lies in one page when pages hold 16 keys
// or more, wherever the window begins); a warp copies its groups into shared memory of its own (cp.async, two groups in
// flight, those of earlier steps' keys before the dependency wait) and works on them alone: scores, masked online softmax
// in float32, P V.  No barrier of the CTA stands in the loop.  The warps' results meet in shared memory, the parts of a
// request in the first CTA of a cluster: every other CTA pushes its accumulator, maximum and sum into an in-box there
// with st.async, which counts the bytes on that CTA's mbarrier (bounded wait, status word), and leaves.  Parts that form no
// cluster go through scratch memory and are added by the CTA that finishes last.  The sum over the parts runs in their
// order either way; a head's sink joins its denominator where the row is finished, once.
//
// Work items, parts, scratch and counters are those of the flash kernel (attention_flash.cuh).
#include "attention_flash.cuh"

#define LA_WARPS 8
#define LA_THREADS (LA_WARPS * 32)
#define LA_GK 16                  // keys per group
#define LA_STAGES 2               // groups in flight per warp
#define LA_ROWS 16                // rows of a CTA
#define LA_LOG2E 1.4426950408889634f

static __device__ int g_la_status = 0;

struct LaArgs {
  const __nv_bfloat16* q; long q_stride;
  const __nv_bfloat16* pages; const int* block_tables; int max_blocks;
  const int* items; __nv_bfloat16* out;
  float* part_acc; float* part_ml; int part_rows;
  int* counters; float scale_log2; int window, H, D, v_pad, page_size;
  const float* sinks;
};

template <int DT> struct LaShape {
  static constexpr int LD = DT + 8;                                   // padded row, in elements
  static constexpr int GROUP_BYTES = LA_GK * LD * 2;
  static constexpr int WARP_BYTES = LA_STAGES * GROUP_BYTES;          // (holds the warp's float32 result [16][DT] at the end)
  static constexpr int Q_BYTES = LA_ROWS * LD * 2;
  static constexpr int BYTES = Q_BYTES + LA_WARPS * WARP_BYTES + LA_WARPS * LA_ROWS * 2 * 4;
  static_assert(WARP_BYTES >= LA_ROWS * DT * 4, "a warp's result fits its stages");
};

__device__ __forceinline__ void la_cp16(void* smem, const void* gmem, bool valid) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(smem);
  const int bytes = valid ? 16 : 0;                 // 0: nothing is read, the 16 bytes are zeroed
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" :: "r"(a), "l"(gmem), "r"(bytes));
}

template <bool CL, int DT>
__global__ void __launch_bounds__(LA_THREADS, 1)
latent_decode_kernel(LaArgs A) {
  using S = LaShape<DT>;
  constexpr int LD = S::LD;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(smem_raw);
  unsigned char* stages = smem_raw + S::Q_BYTES;
  float* s_m = reinterpret_cast<float*>(stages + LA_WARPS * S::WARP_BYTES);     // [warps][16] maxima
  float* s_l = s_m + LA_WARPS * LA_ROWS;                                        // [warps][16] sums
  float* inbox = s_l + LA_WARPS * LA_ROWS;          // CL: [parts - 1][16 v_pad accumulators, then 16 (max, sum)]
  __shared__ uint64_t merge_bar;
  __shared__ int s_abort, s_last;
  pdl_launch_dependents();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int H = A.H, D = A.D, v_pad = A.v_pad, window = A.window, page_size = A.page_size;

  // the work lists come from the host's copy, not from a kernel
  const int* it = A.items + (size_t)blockIdx.x * FA_ITEM_INTS;
  const int req = it[0], q0 = it[1], part = it[4], n_splits = it[5], split = it[6];
  int kv_lo = it[2], kv_hi_item = it[3];
  const int row0 = it[7], q_len = it[8], ctx = it[9];
  const int ntok = min(FA_BM / H, q_len - q0);
  const int first_row = blockIdx.y * LA_ROWS;       // this CTA's rows among the item's (row = token H + head)
  const int nrows = min(LA_ROWS, ntok * H - first_row);
  if (nrows <= 0) { pdl_wait(); return; }           // (the same for every CTA of a cluster)
  if constexpr (CL) {
    if (tid == 0) {
      fa_bar_init(&merge_bar, 1);
      s_abort = 0;
      asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
    }
    asm volatile("barrier.cluster.arrive.release.aligned;\n" ::: "memory");     // looked for when the own part is done
  }
  const int first_pos = ctx + q0;
  if (n_splits > 0) {
    const int total = ctx + q_len;
    const int lo = window > 0 ? max(0, ctx - window + 1) / LA_GK * LA_GK : 0;
    const int per = ((total - lo + n_splits - 1) / n_splits + LA_GK - 1) / LA_GK * LA_GK;
    kv_lo = lo + split * per;
    kv_hi_item = min(total, kv_lo + per);
  }
  const int kv_end = min(kv_hi_item, first_pos + ntok);
  int kv_begin = max(kv_lo, 0);
  if (window > 0) kv_begin = max(kv_begin, first_pos - window + 1);
  const int g_first = kv_begin / LA_GK * LA_GK;     // the groups' first key
  const int n_groups = kv_end > kv_begin ? (kv_end - g_first + LA_GK - 1) / LA_GK : 0;

  const int* __restrict__ table = A.block_tables + (size_t)req * A.max_blocks;
  const int page_shift = (page_size & (page_size - 1)) == 0 ? __ffs(page_size) - 1 : -1;
  const size_t page_stride = (size_t)page_size * D;
  unsigned char* my_stages = stages + (size_t)warp * S::WARP_BYTES;
  const int ch = lane & 15, rsub = lane >> 4;       // this lane's 16-byte pieces of a row: ch, ch + 16; its rows rsub, rsub + 2, ...
  const int chunks = D >> 3;
  auto issue = [&](int gidx, int st) {
    const int j0 = g_first + gidx * LA_GK;
    unsigned char* dst = my_stages + (size_t)st * S::GROUP_BYTES;
    const bool one_page = page_shift >= 4;
    const __nv_bfloat16* base = A.pages;
    if (one_page) base += (size_t)__ldg(table + (j0 >> page_shift)) * page_stride + (size_t)(j0 & (page_size - 1)) * D;
#pragma unroll
    for (int i = 0; i < LA_GK / 2; ++i) {
      const int row = rsub + 2 * i, j = j0 + row;
      const bool ok = j >= kv_begin && j < kv_end;
      const __nv_bfloat16* src = A.pages;
      if (ok) {
        if (one_page) src = base + (size_t)row * D;
        else {
          const int blk = page_shift >= 0 ? j >> page_shift : j / page_size;
          src = A.pages + (size_t)__ldg(table + blk) * page_stride + (size_t)(j - blk * page_size) * D;
        }
      }
#pragma unroll
      for (int cb = 0; cb < (DT + 127) / 128; ++cb) {
        const int c8 = cb * 16 + ch;
        const bool there = ok && c8 < chunks;        // (channels behind the row's own count as zeros)
        if (c8 < DT / 8) la_cp16(dst + row * (LD * 2) + c8 * 16, there ? src + c8 * 8 : A.pages, there);
      }
    }
  };

  // ---- the first groups: those of earlier steps' keys at once, the rest after the wait ------------------------
  bool early[LA_STAGES];
#pragma unroll
  for (int s = 0; s < LA_STAGES; ++s) {
    const int gidx = warp + s * LA_WARPS;
    early[s] = gidx < n_groups && g_first + (gidx + 1) * LA_GK <= ctx;
    if (early[s]) issue(gidx, s);
  }
  pdl_wait();
#pragma unroll
  for (int s = 0; s < LA_STAGES; ++s) {
    const int gidx = warp + s * LA_WARPS;
    if (!early[s] && gidx < n_groups) issue(gidx, s);
    cp_async_commit();                              // one commit per stage, issued or not: the waits below count them
  }
  for (int e = tid; e < LA_ROWS * (DT / 8); e += LA_THREADS) {
    const int r = e / (DT / 8), c8 = e % (DT / 8);
    uint4 v = make_uint4(0, 0, 0, 0);
    if (r < nrows && c8 < chunks) {
      const int ti = (first_row + r) / H, h = (first_row + r) - ti * H;
      v = __ldcg(reinterpret_cast<const uint4*>(A.q + (size_t)(row0 + q0 + ti) * A.q_stride + (size_t)h * D) + c8);
    }
    *reinterpret_cast<uint4*>(sq + r * LD + c8 * 8) = v;
  }
  __syncthreads();

  // ---- this warp's groups --------------------------------------------------------------------------------------
  const int g = lane >> 2, c = lane & 3;
  const int pos_lo = first_pos + (first_row + g) / H, pos_hi = first_pos + (first_row + g + 8) / H;
  float m_lo = -INFINITY, m_hi = -INFINITY, l_lo = 0.f, l_hi = 0.f;
  float o[DT / 8][4];
#pragma unroll
  for (int i = 0; i < DT / 8; ++i) { o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f; }
  int st = 0;
  for (int gidx = warp; gidx < n_groups; gidx += LA_WARPS) {
    cp_async_wait<LA_STAGES - 1>();
    __syncwarp();
    const int j0 = g_first + gidx * LA_GK;
    const __nv_bfloat16* tk = reinterpret_cast<const __nv_bfloat16*>(my_stages + (size_t)st * S::GROUP_BYTES);
    float s[2][2][4];                               // [even, odd steps of k][8 keys][fragment]: two chains of products
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int j = 0; j < 2; ++j) s[i][j][0] = s[i][j][1] = s[i][j][2] = s[i][j][3] = 0.f;
#pragma unroll
    for (int ks = 0; ks < DT / 16; ++ks) {           // (no condition on the row's own channels: the loads of many steps stay in flight)
      uint32_t a[4], b[4];
      ldsm_x4(a, sq + (lane & 15) * LD + ks * 16 + (lane >> 4) * 8);
      ldsm_x4(b, tk + ((lane >> 4) * 8 + (lane & 7)) * LD + ks * 16 + ((lane >> 3) & 1) * 8);
      fa_mma(s[ks & 1][0], a, b[0], b[1]);
      fa_mma(s[ks & 1][1], a, b[2], b[3]);
    }
    float p[2][4];
    float mx_lo = -INFINITY, mx_hi = -INFINITY;
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int key = j0 + j * 8 + 2 * c + e;
        const bool in = key >= kv_begin && key < kv_end;
        const bool ok_lo = in && key <= pos_lo && (window <= 0 || key > pos_lo - window);
        const bool ok_hi = in && key <= pos_hi && (window <= 0 || key > pos_hi - window);
        p[j][e] = ok_lo ? (s[0][j][e] + s[1][j][e]) * A.scale_log2 : -INFINITY;
        p[j][2 + e] = ok_hi ? (s[0][j][2 + e] + s[1][j][2 + e]) * A.scale_log2 : -INFINITY;
        mx_lo = fmaxf(mx_lo, p[j][e]);
        mx_hi = fmaxf(mx_hi, p[j][2 + e]);
      }
    mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 1));
    mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 2));
    mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 1));
    mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 2));
    const float mn_lo = fmaxf(m_lo, mx_lo), mn_hi = fmaxf(m_hi, mx_hi);
    const float base_lo = mn_lo == -INFINITY ? 0.f : mn_lo, base_hi = mn_hi == -INFINITY ? 0.f : mn_hi;
    const float al_lo = exp2f(m_lo - base_lo), al_hi = exp2f(m_hi - base_hi);
    m_lo = mn_lo; m_hi = mn_hi;
    float sum_lo = 0.f, sum_hi = 0.f;
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        p[j][e] = exp2f(p[j][e] - base_lo);
        p[j][2 + e] = exp2f(p[j][2 + e] - base_hi);
        sum_lo += p[j][e];
        sum_hi += p[j][2 + e];
      }
    l_lo = l_lo * al_lo + sum_lo;                   // (this lane's share; the lanes of a row meet after the loop)
    l_hi = l_hi * al_hi + sum_hi;
    uint32_t pa[4] = {pack_bf16(p[0][0], p[0][1]), pack_bf16(p[0][2], p[0][3]), pack_bf16(p[1][0], p[1][1]), pack_bf16(p[1][2], p[1][3])};
#pragma unroll
    for (int dp = 0; dp < DT / 16; ++dp) {
      uint32_t b[4];
      ldsm_x4_t(b, tk + (((lane >> 3) & 1) * 8 + (lane & 7)) * LD + dp * 16 + (lane >> 4) * 8);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        o[2 * dp][e] *= e < 2 ? al_lo : al_hi;
        o[2 * dp + 1][e] *= e < 2 ? al_lo : al_hi;
      }
      fa_mma(o[2 * dp], pa, b[0], b[1]);
      fa_mma(o[2 * dp + 1], pa, b[2], b[3]);
    }
    __syncwarp();                                   // every lane is done with the stage before it is filled again
    const int nxt = gidx + LA_STAGES * LA_WARPS;
    if (nxt < n_groups) issue(nxt, st);
    cp_async_commit();
    st = st + 1 == LA_STAGES ? 0 : st + 1;
  }
  cp_async_wait<0>();
  l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 1);
  l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 2);
  l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 1);
  l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 2);
  __syncwarp();

  // ---- the warps' results meet (each in its own stages' memory first) -----------------------------------------------
  const int used = min(LA_WARPS, n_groups);         // warps that had a group
  float* mine = reinterpret_cast<float*>(my_stages);                  // [16][v_pad]
  if (warp < used) {
#pragma unroll
    for (int i = 0; i < DT / 8; ++i) {
      if (i * 8 < v_pad) {
        if (g < nrows) *reinterpret_cast<float2*>(mine + g * v_pad + i * 8 + 2 * c) = make_float2(o[i][0], o[i][1]);
        if (g + 8 < nrows) *reinterpret_cast<float2*>(mine + (g + 8) * v_pad + i * 8 + 2 * c) = make_float2(o[i][2], o[i][3]);
      }
    }
    if (c == 0) {
      s_m[warp * LA_ROWS + g] = m_lo; s_m[warp * LA_ROWS + g + 8] = m_hi;
      s_l[warp * LA_ROWS + g] = l_lo; s_l[warp * LA_ROWS + g + 8] = l_hi;
    }
  }
  __syncthreads();
  uint32_t crank = 0, box = 0, bar = 0;
  const int per_box = LA_ROWS * (v_pad + 2);
  if constexpr (CL) {
    asm volatile("barrier.cluster.wait.acquire.aligned;\n" ::: "memory");     // (arrived at the top: the barrier exists)
    crank = cluster_cta_rank();
    if (crank != 0) {
      box = cluster_map_shared(inbox + (size_t)(crank - 1) * per_box, 0);
      bar = cluster_map_shared(&merge_bar, 0);
    }
  }
  const int v4 = v_pad >> 2;
  auto store_row = [&](int r, int d4, float4 acc, float l, float mb) {
    const int ti = (first_row + r) / H, h = (first_row + r) - ti * H;
    if (A.sinks) l += exp2f(A.sinks[h] * LA_LOG2E - mb);              // the sink's share of the denominator
    const float inv = l > 0.f ? 1.f / l : 0.f;
    uint2 u;
    u.x = pack_bf16(acc.x * inv, acc.y * inv);
    u.y = pack_bf16(acc.z * inv, acc.w * inv);
    *reinterpret_cast<uint2*>(A.out + (size_t)(row0 + q0 + ti) * ((size_t)H * D) + (size_t)h * D + 4 * d4) = u;
  };
  for (int e = tid; e < nrows * v4; e += LA_THREADS) {
    const int r = e / v4, d4 = e - r * v4;
    float m = -INFINITY;
    for (int w = 0; w < used; ++w) m = fmaxf(m, s_m[w * LA_ROWS + r]);
    const float mb = m == -INFINITY ? 0.f : m;
    float l = 0.f;
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int w = 0; w < LA_WARPS; ++w) {
      if (w < used) {
        const float wgt = exp2f(s_m[w * LA_ROWS + r] - mb);
        const float4 v = *reinterpret_cast<const float4*>(stages + (size_t)w * S::WARP_BYTES + ((size_t)r * v_pad + 4 * d4) * 4);
        l += wgt * s_l[w * LA_ROWS + r];
        acc.x += wgt * v.x; acc.y += wgt * v.y; acc.z += wgt * v.z; acc.w += wgt * v.w;
      }
    }
    if constexpr (CL) {
      if (crank != 0) {
        // into the first CTA's in-box: the accumulator, and once per row the maximum and the sum
        asm volatile("st.async.weak.shared::cluster.mbarrier::complete_tx::bytes.v4.b32 [%0], {%1, %2, %3, %4}, [%5];\n"
                     :: "r"(box + 4u * (uint32_t)(r * v_pad + 4 * d4)), "r"(__float_as_uint(acc.x)), "r"(__float_as_uint(acc.y)),
                        "r"(__float_as_uint(acc.z)), "r"(__float_as_uint(acc.w)), "r"(bar) : "memory");
        if (d4 == 0) {
          const uint32_t at = box + 4u * (uint32_t)(LA_ROWS * v_pad + 2 * r);
          asm volatile("st.async.weak.shared::cluster.mbarrier::complete_tx::bytes.b32 [%0], %1, [%2];\n"
                       :: "r"(at), "r"(__float_as_uint(m)), "r"(bar) : "memory");
          asm volatile("st.async.weak.shared::cluster.mbarrier::complete_tx::bytes.b32 [%0], %1, [%2];\n"
                       :: "r"(at + 4u), "r"(__float_as_uint(l)), "r"(bar) : "memory");
        }
      } else {
        // this CTA's own sums stay with the thread that formed them: it is the one that merges this element below
        *reinterpret_cast<float4*>(stages + ((size_t)r * v_pad + 4 * d4) * 4) = acc;
      }
    } else if (part < 0) {
      store_row(r, d4, acc, l, mb);
    } else {
      const size_t slot = (size_t)part * A.part_rows + first_row + r;
      *reinterpret_cast<float4*>(A.part_acc + slot * D + 4 * d4) = acc;
      if (d4 == 0) { A.part_ml[2 * slot] = m; A.part_ml[2 * slot + 1] = l; }
    }
  }
  if constexpr (CL) {
    if (crank != 0) return;
    const int parts = (int)cluster_num_ctas();      // = n_splits, at most 8
    if (tid == 0) {
      const uint32_t bytes = (uint32_t)(parts - 1) * (uint32_t)(nrows * v_pad + 2 * nrows) * 4u;
      asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;\n" :: "r"(fa_smem(&merge_bar)), "r"(bytes) : "memory");
    }
    bool landed = false;
    for (uint32_t i = 0; i < FA_WAIT_LIMIT && !landed; ++i) {
      uint32_t ok;
      asm volatile("{\n\t.reg .pred p;\n\tmbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\tselp.b32 %0, 1, 0, p;\n\t}\n"
                   : "=r"(ok) : "r"(fa_smem(&merge_bar)), "r"(0u) : "memory");
      landed = ok != 0;
    }
    if (!landed) { atomicCAS(&g_la_status, 0, 1); return; }           // bounded: the word says so, nothing is written
    for (int e = tid; e < nrows * v4; e += LA_THREADS) {
      const int r = e / v4, d4 = e - r * v4;
      // this CTA's own maximum and sum once more (few numbers, in shared memory)
      float m0 = -INFINITY;
      for (int w = 0; w < used; ++w) m0 = fmaxf(m0, s_m[w * LA_ROWS + r]);
      const float mb0 = m0 == -INFINITY ? 0.f : m0;
      float l0 = 0.f;
      for (int w = 0; w < used; ++w) l0 += exp2f(s_m[w * LA_ROWS + r] - mb0) * s_l[w * LA_ROWS + r];
      float m = m0;
      for (int sp = 1; sp < parts; ++sp) m = fmaxf(m, inbox[(size_t)(sp - 1) * per_box + LA_ROWS * v_pad + 2 * r]);
      const float mb = m == -INFINITY ? 0.f : m;
      const float w0 = exp2f(m0 - mb);
      float4 acc = *reinterpret_cast<const float4*>(stages + ((size_t)r * v_pad + 4 * d4) * 4);
      acc.x *= w0; acc.y *= w0; acc.z *= w0; acc.w *= w0;
      float l = l0 * w0;
      for (int sp = 1; sp < parts; ++sp) {          // in the order of the parts
        const float* b = inbox + (size_t)(sp - 1) * per_box;
        const float wgt = exp2f(b[LA_ROWS * v_pad + 2 * r] - mb);
        const float4 v = *reinterpret_cast<const float4*>(b + r * v_pad + 4 * d4);
        l += wgt * b[LA_ROWS * v_pad + 2 * r + 1];
        acc.x += wgt * v.x; acc.y += wgt * v.y; acc.z += wgt * v.z; acc.w += wgt * v.w;
      }
      store_row(r, d4, acc, l, mb);
    }
  } else if (part >= 0 && n_splits > 0) {
    // ---- the CTA that finishes a request's last part adds the parts ----------------------------------------------------
    const int first = part - split;
    __threadfence();                                // this CTA's part is visible before it is counted
    __syncthreads();
    if (tid == 0) {
      int* counter = A.counters + (size_t)first * gridDim.y + blockIdx.y;
      const int done = atomicAdd(counter, 1);
      s_last = (done == n_splits - 1);
      if (s_last) *counter = 0;                     // ready for the next launch
    }
    __syncthreads();
    if (s_last) {
      __threadfence();
      for (int e = tid; e < nrows * v4; e += LA_THREADS) {
        const int r = e / v4, d4 = e - r * v4;
        const size_t slot0 = (size_t)first * A.part_rows + first_row + r;
        float m = -INFINITY;
#pragma unroll 4
        for (int sp = 0; sp < n_splits; ++sp) m = fmaxf(m, __ldcg(A.part_ml + 2 * (slot0 + (size_t)sp * A.part_rows)));
        const float mb = m == -INFINITY ? 0.f : m;
        float l = 0.f;
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
        for (int sp = 0; sp < n_splits; ++sp) {
          const size_t slot = slot0 + (size_t)sp * A.part_rows;
          const float2 ml = __ldcg(reinterpret_cast<const float2*>(A.part_ml + 2 * slot));
          const float4 v = __ldcg(reinterpret_cast<const float4*>(A.part_acc + slot * D + 4 * d4));
          const float wgt = exp2f(ml.x - mb);
          l += wgt * ml.y;
          acc.x += wgt * v.x; acc.y += wgt * v.y; acc.z += wgt * v.z; acc.w += wgt * v.w;
        }
        store_row(r, d4, acc, l, mb);
      }
    }
  }
}

#define LA_SMEM_LIMIT (226 * 1024)                  // (an SM has 227 KB; the kernel's static variables take some)

template <int DT>
static int la_smem(int v_pad, int parts) { return LaShape<DT>::BYTES + (parts > 1 ? (parts - 1) * LA_ROWS * (v_pad + 2) * 4 : 0); }
static int la_smem_of(int D, int v_pad, int parts) {
  return D <= 64 ? la_smem<64>(v_pad, parts) : D <= 128 ? la_smem<128>(v_pad, parts) : D <= 192 ? la_smem<192>(v_pad, parts) : la_smem<256>(v_pad, parts);
}

// The most parts of a request (8, 4, 2 or 1) whose in-boxes fit beside the warps' memory, for cache rows of D channels;
// 0 where the kernel does not take the size.
extern "C" int qe_latent_decode_max_parts(int D) {
  if (D < 16 || D > 256 || D % 16) return 0;
  for (int s = 8; s > 1; s >>= 1)
    if (la_smem_of(D, D, s) <= LA_SMEM_LIMIT) return s;
  return 1;
}

template <bool CL, int DT>
static int launch_latent_decode(const LaArgs& A, int n_items, int row_tiles, int cluster, cudaStream_t stream) {
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel<CL, DT>, cudaFuncAttributeMaxDynamicSharedMemorySize, LA_SMEM_LIMIT);
    if (e != cudaSuccess) QE_REFUSE("latent_decode: shared memory: %s", cudaGetErrorString(e));
    configured = true;
  }
  const int smem = la_smem<DT>(A.v_pad, CL ? cluster : 1);
  if (smem > LA_SMEM_LIMIT) QE_REFUSE("latent_decode: %d parts of %d channels do not fit shared memory", cluster, A.v_pad);
  const dim3 grid(n_items, row_tiles);
  if (CL) qe_launch_cluster(latent_decode_kernel<CL, DT>, grid, dim3(LA_THREADS), smem, stream, (unsigned)cluster, A);
  else qe_launch(latent_decode_kernel<CL, DT>, grid, dim3(LA_THREADS), smem, stream, A);
  QE_CHECK_LAUNCH("latent_decode");
  return 0;
}

// q [T, H D] (rows may be strided), pages [pages, page, D], out [T, H D] (the first v_dim channels of every head, rounded up to a
// multiple of 16, are written); items and scratch as for the flash kernel, max_rows the most rows of an item.  cluster: the
// number of parts of every request (2, 4 or 8) when the items are exactly those parts in order, else 0: parts then need the
// counters (one int per part and 16 rows, zero before the first use).
extern "C" int qe_latent_decode(const void* q, long q_stride, const void* pages, const int* block_tables, int max_blocks,
                                const int* items, int n_items, void* out, float* part_acc, float* part_ml, int part_rows,
                                int* counters, int max_rows, int cluster, float scale, int window, int H, int D, int v_dim,
                                int page_size, const float* sinks, cudaStream_t stream) {
  if (n_items <= 0) return 0;
  if (D < 16 || D > 256 || D % 16 || H < 1 || H > FA_BM) QE_REFUSE("latent_decode: %d heads over cache rows of %d channels", H, D);
  if (v_dim < 1 || v_dim > D || max_rows < 1 || max_rows > FA_BM) QE_REFUSE("latent_decode: values of %d channels, %d rows", v_dim, max_rows);
  if ((((uintptr_t)q | (uintptr_t)pages | (uintptr_t)out | (uintptr_t)part_acc | (uintptr_t)part_ml) & 15) || q_stride % 8)
    QE_REFUSE("latent_decode: operands must be 16-byte aligned");
  if (part_acc && counters == nullptr && !cluster) QE_REFUSE("latent_decode: parts need the counters");
  if (cluster && ((cluster != 2 && cluster != 4 && cluster != 8) || n_items % cluster))
    QE_REFUSE("latent_decode: %d items cannot form clusters of %d", n_items, cluster);
  const LaArgs A{(const __nv_bfloat16*)q, q_stride, (const __nv_bfloat16*)pages, block_tables, max_blocks, items, (__nv_bfloat16*)out,
                 part_acc, part_ml, part_rows, counters, scale * LA_LOG2E, window, H, D, (v_dim + 15) / 16 * 16, page_size, sinks};
  const int row_tiles = (max_rows + LA_ROWS - 1) / LA_ROWS;
#define LA_GO(DT) return cluster ? launch_latent_decode<true, DT>(A, n_items, row_tiles, cluster, stream) \
                                 : launch_latent_decode<false, DT>(A, n_items, row_tiles, 0, stream)
  if (D <= 64) LA_GO(64);
  if (D <= 128) LA_GO(128);
  if (D <= 192) LA_GO(192);
  LA_GO(256);
#undef LA_GO
}

// The status word of the bounded wait for the pushed parts (0 = fine).
extern "C" int qe_latent_decode_status() {
  int v = 0;
  cudaMemcpyFromSymbol(&v, g_la_status, sizeof(int));
  return v;
}
extern "C" void qe_latent_decode_clear_status() {
  int v = 0;
  cudaMemcpyToSymbol(g_la_status, &v, sizeof(int));
}
