// The two products of routed experts without a gate for steps of a few tokens (decoded tokens), bfloat16: every weight of
// the experts that are used is read once, in the manner of the weight-streaming product of the dense layers
// (gemm_small_m.cuh): the weight rows ride the M dimension of mma.sync.m16n8k16, so a 16-byte load of a weight row feeds
// the tensor core directly, and the expert's tokens ride its N dimension.
//
//   qe_moe_small_up     act[p, :] = f(W_up_e x_t) for the pair p = (t, e) in sorted order
//   qe_moe_small_down   y[p, :] = W_down_e act[p, :], float32
//
// One CTA of 8 warps owns 16 weight rows of one expert; the warps split K and their sums are added in their order, so a
// row's bits depend on K alone.  A CTA whose expert has no token leaves; an expert with more tokens than a tile holds is
// walked tile by tile (its weights then come from L2).
#include "gemm_small_m.cuh"

#define MS_WARPS 8
#define MS_THREADS (MS_WARPS * 32)

// UP: rows gathered from x by pair / top, activation, bfloat16 out [P, N]; else rows are x[p], float32 out [P, N].
// MT: tiles of 8 tokens at a time.
template <int MT, bool UP>
__global__ void __launch_bounds__(MS_THREADS)
moe_small_kernel(const __nv_bfloat16* __restrict__ x, const __nv_bfloat16* __restrict__ w, const int* __restrict__ offsets,
                 const int* __restrict__ sorted_pair, void* __restrict__ out_, int N, int K, int k_per_warp, int top, int act,
                 const float* __restrict__ pair_w, int early) {
  __shared__ float red[MS_WARPS * 16 * 8 * MT];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, c = lane & 3;
  const int e = blockIdx.y, n0 = blockIdx.x * 16;
  const __nv_bfloat16* we = w + (size_t)e * N * K;
  const __nv_bfloat16* w0 = we + (size_t)min(n0 + g, N - 1) * K;          // clamped; discarded at the store
  const __nv_bfloat16* w1 = we + (size_t)min(n0 + g + 8, N - 1) * K;
  const int kbeg = warp * k_per_warp, kend = min(K, kbeg + k_per_warp);
  const uint4 zero = make_uint4(0, 0, 0, 0);
  auto load_chunk = [&](int k0) {
    GsmChunk ch;
    const int ka = k0 + 8 * c, kb = k0 + 32 + 8 * c;
    ch.a0 = ka < kend ? ld_stream16(w0 + ka) : zero;
    ch.b0 = ka < kend ? ld_stream16(w1 + ka) : zero;
    ch.a1 = kb < kend ? ld_stream16(w0 + kb) : zero;
    ch.b1 = kb < kend ? ld_stream16(w1 + kb) : zero;
    return ch;
  };
  // Where nearly every expert is used, the first weights are on their way before the wait for the kernel that says so.
  GsmChunk c0{zero, zero, zero, zero}, c1 = c0;
  if (early) { c0 = load_chunk(kbeg); c1 = load_chunk(kbeg + 64); }
  pdl_launch_dependents();
  pdl_wait();
  const int first = __ldcg(offsets + e), rows = __ldcg(offsets + e + 1) - first;
  if (rows <= 0) return;
  if (!early) { c0 = load_chunk(kbeg); c1 = load_chunk(kbeg + 64); }
  for (int m0 = 0; m0 < rows; m0 += 8 * MT) {
    if (m0 > 0) { c0 = load_chunk(kbeg); c1 = load_chunk(kbeg + 64); }
    const __nv_bfloat16* xr[MT];
#pragma unroll
    for (int t = 0; t < MT; ++t) {
      const int m = m0 + t * 8 + g;
      xr[t] = m >= rows ? nullptr
              : x + (size_t)(UP ? __ldcg(sorted_pair + first + m) / top : first + m) * K;
    }
    float acc[MT][4];
#pragma unroll
    for (int t = 0; t < MT; ++t) acc[t][0] = acc[t][1] = acc[t][2] = acc[t][3] = 0.f;
    auto load_x = [&](int t, int k) {
      return xr[t] != nullptr && k < kend ? __ldcg(reinterpret_cast<const uint4*>(xr[t] + k)) : zero;
    };
    auto compute = [&](const GsmChunk& ch, int k0) {
      const int ka = k0 + 8 * c, kb = k0 + 32 + 8 * c;
#pragma unroll
      for (int t = 0; t < MT; ++t) {
        const uint4 xa = load_x(t, ka), xb = load_x(t, kb);
        mma_bf16_16816(acc[t], ch.a0.x, ch.b0.x, ch.a0.y, ch.b0.y, xa.x, xa.y);
        mma_bf16_16816(acc[t], ch.a0.z, ch.b0.z, ch.a0.w, ch.b0.w, xa.z, xa.w);
        mma_bf16_16816(acc[t], ch.a1.x, ch.b1.x, ch.a1.y, ch.b1.y, xb.x, xb.y);
        mma_bf16_16816(acc[t], ch.a1.z, ch.b1.z, ch.a1.w, ch.b1.w, xb.z, xb.w);
      }
    };
    for (int k0 = kbeg; k0 < kend; k0 += 128) {
      const GsmChunk d0 = load_chunk(k0 + 128);
      compute(c0, k0);
      const GsmChunk d1 = load_chunk(k0 + 192);
      compute(c1, k0 + 64);
      c0 = d0;
      c1 = d1;
    }
    constexpr int MW = 8 * MT;
    float* mine = red + (size_t)warp * 16 * MW;
#pragma unroll
    for (int t = 0; t < MT; ++t) {
      mine[g * MW + t * 8 + 2 * c] = acc[t][0];
      mine[g * MW + t * 8 + 2 * c + 1] = acc[t][1];
      mine[(g + 8) * MW + t * 8 + 2 * c] = acc[t][2];
      mine[(g + 8) * MW + t * 8 + 2 * c + 1] = acc[t][3];
    }
    __syncthreads();
    for (int i = threadIdx.x; i < 16 * MW; i += MS_THREADS) {
      const int m = i >> 4, r = i & 15, n = n0 + r;
      if (m0 + m < rows && n < N) {
        float s = 0.f;
#pragma unroll
        for (int wi = 0; wi < MS_WARPS; ++wi) s += red[((size_t)wi * 16 + r) * MW + m];
        const size_t at = (size_t)(first + m0 + m) * N + n;
        if constexpr (UP) {
          const float pw = pair_w ? pair_w[sorted_pair[first + m0 + m]] : 1.f;
          ((__nv_bfloat16*)out_)[at] = __float2bfloat16_rn(act_exact(s * pw, act));
        } else {
          ((float*)out_)[at] = s;
        }
      }
    }
    if (m0 + MW < rows) __syncthreads();
  }
}

template <bool UP>
static int moe_small_launch(const void* x, const void* w, const int* offsets, const int* sorted_pair, void* out, int T, int P, int E,
                            int N, int K, int top, int act, const float* pair_w, cudaStream_t stream) {
  if (P <= 0) return 0;
  if (T < 1 || T > 64 || K < 8 || K % 8) QE_REFUSE("moe_small: %d tokens, K = %d", T, K);
  if (E < 1 || E > 65535) QE_REFUSE("moe_small: %d experts", E);
  if (((uintptr_t)x | (uintptr_t)w) & 15) QE_REFUSE("moe_small: operands must be 16-byte aligned");
  const int k_per_warp = ((K + MS_WARPS - 1) / MS_WARPS + 63) / 64 * 64;
  const dim3 grid((N + 15) / 16, E);
  const int early = E <= P ? 1 : 0;
#define MS_GO(MT) qe_launch(moe_small_kernel<MT, UP>, grid, dim3(MS_THREADS), 0, stream, (const __nv_bfloat16*)x, (const __nv_bfloat16*)w, \
                            offsets, sorted_pair, out, N, K, k_per_warp, top, act, pair_w, early)
  if (T <= 8) MS_GO(1);
  else if (T <= 16) MS_GO(2);
  else MS_GO(4);
#undef MS_GO
  QE_CHECK_LAUNCH("moe_small");
  return 0;
}

// T: the step's tokens (at most 64; an expert has at most so many rows).  The rest as qe_moe_up and qe_moe_down (one share).
extern "C" int qe_moe_small_up(const void* x, const void* w, const int* offsets, const int* sorted_pair, void* act_out, int T, int P,
                               int E, int I, int K, int top, int act, const float* pair_w, cudaStream_t stream) {
  if (act < 0 || act > QE_ACT_MAX || top < 1) QE_REFUSE("moe_small_up: activation %d, %d choices", act, top);
  return moe_small_launch<true>(x, w, offsets, sorted_pair, act_out, T, P, E, I, K, top, act, pair_w, stream);
}
extern "C" int qe_moe_small_down(const void* act_in, const void* w, const int* offsets, float* y, int T, int P, int E, int N, int K,
                                 cudaStream_t stream) {
  return moe_small_launch<false>(act_in, w, offsets, nullptr, (void*)y, T, P, E, N, K, 1, 0, nullptr, stream);
}
