// RMS norms of whole rows that do more than one thing in a pass, the row in registers between the sum of squares and the
// scaling:
//
//   qe_add_rmsnorm_pair    the residual stream of an arrangement whose two sublayers read the same stream through norms
//                          of their own: x = resid + delta_a + delta_b;  out1 = x / rms(x) * w1,  out2 = x / rms(x) * w2,
//                          resid = x + bias (a bias of the sublayers' results rides on the stream's write)
//   qe_group_norm_gate     a recurrent mixer's output, normed in groups and gated: y = x / den (a divisor per group), or
//                          y = x * g(gate) where the gate comes ahead of the norm;  out = y / rms(y) * w * g(gate) * scale
//
// Float32 arithmetic, results rounded once.  The order of every sum depends on the sizes alone.
#include "common.cuh"
#include <math.h>

template <typename T> __device__ __forceinline__ void nr_ld4(const T* p, float (&f)[4]);
template <> __device__ __forceinline__ void nr_ld4<float>(const float* p, float (&f)[4]) {
  const float4 v = *reinterpret_cast<const float4*>(p); f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w; }
template <> __device__ __forceinline__ void nr_ld4<__nv_bfloat16>(const __nv_bfloat16* p, float (&f)[4]) {
  const uint2 r = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
  f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y; }
template <typename T> __device__ __forceinline__ void nr_st4(T* p, const float (&f)[4]);
template <> __device__ __forceinline__ void nr_st4<float>(float* p, const float (&f)[4]) { *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]); }
template <> __device__ __forceinline__ void nr_st4<__nv_bfloat16>(__nv_bfloat16* p, const float (&f)[4]) {
  __nv_bfloat162 lo = __floats2bfloat162_rn(f[0], f[1]), hi = __floats2bfloat162_rn(f[2], f[3]);
  uint2 r;
  r.x = *reinterpret_cast<uint32_t*>(&lo); r.y = *reinterpret_cast<uint32_t*>(&hi);
  *reinterpret_cast<uint2*>(p) = r; }

// Sum over `warps` warps of a CTA (all of it), fixed order; one meeting.
__device__ __forceinline__ float nr_sum(float v, float* red, int warps) {
  v = warp_sum(v);
  if (warps == 1) return v;
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  for (int w = 0; w < warps; ++w) t += red[w];
  return t;
}

// ---------------------------------------------------------------------------------------------------------
struct PairArgs {
  float* resid; const void* da; const void* db; const float* bias;
  const float* w1; const float* w2; void* o1; void* o2; float eps; int H;
};

// NV pieces of four channels a thread
template <typename T, int NV>
__global__ void __launch_bounds__(256) add_rmsnorm_pair_kernel(PairArgs A) {
  __shared__ float red[8];
  pdl_launch_dependents();
  const int H = A.H, warps = blockDim.x >> 5;
  float w1[NV][4], w2[NV][4], b[NV][4];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int h = (i * blockDim.x + threadIdx.x) * 4;
    if (h >= H) continue;
    nr_ld4(A.w1 + h, w1[i]);
    if (A.o2) nr_ld4(A.w2 + h, w2[i]);
    if (A.bias) nr_ld4(A.bias + h, b[i]);
  }
  pdl_wait();
  const size_t row = (size_t)blockIdx.x * H;
  float x[NV][4], a[NV][4], c[NV][4];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int h = (i * blockDim.x + threadIdx.x) * 4;
    if (h >= H) continue;
    nr_ld4(A.resid + row + h, x[i]);
    if (A.da) nr_ld4((const T*)A.da + row + h, a[i]);
    if (A.db) nr_ld4((const T*)A.db + row + h, c[i]);
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int h = (i * blockDim.x + threadIdx.x) * 4;
    if (h >= H) continue;
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      if (A.da) x[i][u] += a[i][u];
      if (A.db) x[i][u] += c[i][u];
      ss = fmaf(x[i][u], x[i][u], ss);
    }
  }
  ss = nr_sum(ss, red, warps);
  const float rstd = rsqrtf(ss / (float)H + A.eps);
  const bool writes = A.da || A.db || A.bias;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int h = (i * blockDim.x + threadIdx.x) * 4;
    if (h >= H) continue;
    float r[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) r[u] = x[i][u] * rstd * w1[i][u];
    nr_st4((T*)A.o1 + row + h, r);
    if (A.o2) {
#pragma unroll
      for (int u = 0; u < 4; ++u) r[u] = x[i][u] * rstd * w2[i][u];
      nr_st4((T*)A.o2 + row + h, r);
    }
    if (writes) {
#pragma unroll
      for (int u = 0; u < 4; ++u) r[u] = A.bias ? x[i][u] + b[i][u] : x[i][u];
      nr_st4(A.resid + row + h, r);
    }
  }
}

// any width, channel by channel
template <typename T>
__global__ void __launch_bounds__(256) add_rmsnorm_pair_plain_kernel(PairArgs A) {
  __shared__ float red[8];
  pdl_launch_dependents();
  pdl_wait();
  const int H = A.H;
  const size_t row = (size_t)blockIdx.x * H;
  float ss = 0.f;
  for (int h = threadIdx.x; h < H; h += blockDim.x) {
    float x = A.resid[row + h];
    if (A.da) x += to_f32(((const T*)A.da)[row + h]);
    if (A.db) x += to_f32(((const T*)A.db)[row + h]);
    A.resid[row + h] = x;
    ss = fmaf(x, x, ss);
  }
  ss = nr_sum(ss, red, blockDim.x >> 5);
  const float rstd = rsqrtf(ss / (float)H + A.eps);
  for (int h = threadIdx.x; h < H; h += blockDim.x) {
    const float x = A.resid[row + h];
    ((T*)A.o1)[row + h] = from_f32<T>(x * rstd * A.w1[h]);
    if (A.o2) ((T*)A.o2)[row + h] = from_f32<T>(x * rstd * A.w2[h]);
    if (A.bias) A.resid[row + h] = x + A.bias[h];
  }
}

extern "C" int qe_add_rmsnorm_pair(float* resid, const void* da, const void* db, const float* bias, const float* w1, const float* w2,
                                   float eps, void* o1, void* o2, int T, int H, int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (dtype != QE_DTYPE_F32 && dtype != QE_DTYPE_BF16) QE_REFUSE("add_rmsnorm_pair: unknown dtype %d", dtype);
  if (o2 && !w2) QE_REFUSE("add_rmsnorm_pair: a second output needs its weights");
  PairArgs A{resid, da, db, bias, w1, w2, o1, o2, eps, H};
  const bool aligned = H % 4 == 0 && (((uintptr_t)resid | (uintptr_t)da | (uintptr_t)db | (uintptr_t)bias | (uintptr_t)w1 | (uintptr_t)w2 |
                                       (uintptr_t)o1 | (uintptr_t)o2) & 15) == 0;
  const int pieces = H / 4;
  const int threads = pieces <= 128 ? (pieces + 31) / 32 * 32 : 256;
  const int nv = aligned ? (pieces + threads - 1) / threads : 99;
#define PAIR(TT) do { \
    if (nv <= 1) qe_launch(add_rmsnorm_pair_kernel<TT, 1>, dim3(T), dim3(threads), 0, stream, A); \
    else if (nv <= 2) qe_launch(add_rmsnorm_pair_kernel<TT, 2>, dim3(T), dim3(threads), 0, stream, A); \
    else if (nv <= 4) qe_launch(add_rmsnorm_pair_kernel<TT, 4>, dim3(T), dim3(threads), 0, stream, A); \
    else if (nv <= 8) qe_launch(add_rmsnorm_pair_kernel<TT, 8>, dim3(T), dim3(threads), 0, stream, A); \
    else qe_launch(add_rmsnorm_pair_plain_kernel<TT>, dim3(T), dim3(256), 0, stream, A); } while (0)
  if (dtype == QE_DTYPE_F32) PAIR(float); else PAIR(__nv_bfloat16);
#undef PAIR
  QE_CHECK_LAUNCH("add_rmsnorm_pair");
  return 0;
}

// ---------------------------------------------------------------------------------------------------------
struct GroupGateArgs {
  const float* x; long ldx; const void* g; long ldg; const float* w; const float* den; void* out; long ldo;
  float eps, scale; int G, D, gate, gate_first, items;      // G groups of D channels; gate 0 none, 1 silu, 2 sigmoid
};
// (bfloat16 results: the hardware's exponential and quotient)
template <typename T> __device__ __forceinline__ float nr_gate(float g, int kind) {
  if (kind == 0) return 1.f;
  const float num = kind == 1 ? g : 1.f;
  return sizeof(T) == 4 ? num / (1.f + expf(-g)) : __fdividef(num, 1.f + __expf(-g));
}

// WPG warps a group (1: eight groups a CTA; else the CTA is one group's), NV pieces of four channels a thread
template <typename T, int WPG, int NV>
__global__ void __launch_bounds__(256) group_norm_gate_kernel(GroupGateArgs A) {
  __shared__ float red[8];
  pdl_launch_dependents();
  const int item = WPG == 1 ? blockIdx.x * 8 + (threadIdx.x >> 5) : blockIdx.x;
  const int tid = WPG == 1 ? threadIdx.x & 31 : threadIdx.x;
  constexpr int TPG = WPG * 32;
  const int D = A.D;
  const int t = item / A.G, gr = item - t * A.G;
  const bool in = item < A.items;
  float wv[NV][4];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int d = (i * TPG + tid) * 4;
    if (in && d < D) nr_ld4(A.w + (size_t)gr * D + d, wv[i]);
  }
  pdl_wait();
  if (!in) return;                                   // (a whole warp; the CTA has one group where its warps meet)
  const float* x = A.x + (size_t)t * A.ldx + (size_t)gr * D;
  const T* g = A.g ? (const T*)A.g + (size_t)t * A.ldg + (size_t)gr * D : nullptr;
  float v[NV][4], gv[NV][4];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int d = (i * TPG + tid) * 4;
    if (d >= D) continue;
    nr_ld4(x + d, v[i]);
    if (g) nr_ld4(g + d, gv[i]);
  }
  const float div = A.den ? A.den[item] : 1.f;
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int d = (i * TPG + tid) * 4;
    if (d >= D) continue;
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      if (g) gv[i][u] = nr_gate<T>(gv[i][u], A.gate);
      if (A.den) v[i][u] = v[i][u] / div;
      if (A.gate_first && g) v[i][u] *= gv[i][u];
      ss = fmaf(v[i][u], v[i][u], ss);
    }
  }
  ss = nr_sum(ss, red, WPG);
  const float rstd = rsqrtf(ss / (float)D + A.eps);
  T* out = (T*)A.out + (size_t)t * A.ldo + (size_t)gr * D;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int d = (i * TPG + tid) * 4;
    if (d >= D) continue;
    float r[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      r[u] = v[i][u] * rstd * wv[i][u];
      if (g && !A.gate_first) r[u] *= gv[i][u];
      r[u] *= A.scale;
    }
    nr_st4(out + d, r);
  }
}

// any size and alignment: a CTA a group, channel by channel
template <typename T>
__global__ void __launch_bounds__(128) group_norm_gate_plain_kernel(GroupGateArgs A) {
  __shared__ float red[4];
  pdl_launch_dependents();
  pdl_wait();
  const int item = blockIdx.x, t = item / A.G, gr = item - t * A.G, D = A.D;
  const float* x = A.x + (size_t)t * A.ldx + (size_t)gr * D;
  const T* g = A.g ? (const T*)A.g + (size_t)t * A.ldg + (size_t)gr * D : nullptr;
  const float div = A.den ? A.den[item] : 1.f;
  auto value = [&](int d) {
    float v = A.den ? x[d] / div : x[d];
    if (A.gate_first && g) v *= nr_gate<T>(to_f32(g[d]), A.gate);
    return v;
  };
  float ss = 0.f;
  for (int d = threadIdx.x; d < D; d += blockDim.x) { const float v = value(d); ss = fmaf(v, v, ss); }
  ss = nr_sum(ss, red, 4);
  const float rstd = rsqrtf(ss / (float)D + A.eps);
  T* out = (T*)A.out + (size_t)t * A.ldo + (size_t)gr * D;
  for (int d = threadIdx.x; d < D; d += blockDim.x) {
    float r = value(d) * rstd * A.w[(size_t)gr * D + d];
    if (g && !A.gate_first) r *= nr_gate<T>(to_f32(g[d]), A.gate);
    out[d] = from_f32<T>(r * A.scale);
  }
}

extern "C" int qe_group_norm_gate(const float* x, long ldx, const void* g, long ldg, const float* w, const float* den, float eps,
                                  void* out, long ldo, float scale, int gate, int gate_first, int T, int G, int D, int dtype,
                                  cudaStream_t stream) {
  if (T <= 0) return 0;
  if (dtype != QE_DTYPE_F32 && dtype != QE_DTYPE_BF16) QE_REFUSE("group_norm_gate: unknown dtype %d", dtype);
  if (G < 1 || D < 1 || (long)T * G > 0x7fffffffL) QE_REFUSE("group_norm_gate: %d groups of %d channels", G, D);
  if (w == nullptr) QE_REFUSE("group_norm_gate: the norm's weights are needed");
  GroupGateArgs A{x, ldx, g, ldg, w, den, out, ldo, eps, scale, G, D, g ? gate : 0, gate_first, T * G};
  const size_t es = dtype == QE_DTYPE_F32 ? 4 : 2;
  const bool aligned = D % 4 == 0 && ldx % 4 == 0 && (!g || ldg % 4 == 0) && ldo % 4 == 0 && (((uintptr_t)x | (uintptr_t)w) & 15) == 0 &&
                       ((uintptr_t)g % (4 * es)) == 0 && ((uintptr_t)out % (4 * es)) == 0;
  const int pieces = D / 4;
  const unsigned one = (unsigned)((A.items + 7) / 8), cta = (unsigned)A.items;
#define GNG(TT) do { \
    if (aligned && pieces <= 32) qe_launch(group_norm_gate_kernel<TT, 1, 1>, dim3(one), dim3(256), 0, stream, A); \
    else if (aligned && pieces <= 64) qe_launch(group_norm_gate_kernel<TT, 1, 2>, dim3(one), dim3(256), 0, stream, A); \
    else if (aligned && pieces <= 128) qe_launch(group_norm_gate_kernel<TT, 4, 1>, dim3(cta), dim3(128), 0, stream, A); \
    else if (aligned && pieces <= 256) qe_launch(group_norm_gate_kernel<TT, 8, 1>, dim3(cta), dim3(256), 0, stream, A); \
    else if (aligned && pieces <= 512) qe_launch(group_norm_gate_kernel<TT, 8, 2>, dim3(cta), dim3(256), 0, stream, A); \
    else if (aligned && pieces <= 1024) qe_launch(group_norm_gate_kernel<TT, 8, 4>, dim3(cta), dim3(256), 0, stream, A); \
    else if (aligned && pieces <= 2048) qe_launch(group_norm_gate_kernel<TT, 8, 8>, dim3(cta), dim3(256), 0, stream, A); \
    else qe_launch(group_norm_gate_plain_kernel<TT>, dim3(cta), dim3(128), 0, stream, A); } while (0)
  if (dtype == QE_DTYPE_F32) GNG(float); else GNG(__nv_bfloat16);
#undef GNG
  QE_CHECK_LAUNCH("group_norm_gate");
  return 0;
}
