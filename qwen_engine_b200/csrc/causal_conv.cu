// Short causal convolutions over time on each channel of a projection, several channels a thread, with what follows them
// in the same kernel:
//
//   u_t = x_t (+ bias)                                    the projected row, its bias added in float32
//   y_t[c] = sum_j w[j][c] u_(t - taps + 1 + j)[c]         u = 0 before the sequence's first token
//
// qe_conv_act:  out = act(y + out_bias), act silu or none, rounded once to the compute type;
// qe_conv_qkv:  y holds the query, key and value heads of attention: the first rot_dims channels of every query and key
//               head turn (pairs (i, i + rot_dims / 2), angle position * inv_freq[i]), queries go to a buffer of their own,
//               keys and values to their slots in the pages.
//
// The state of a request is its last taps - 1 rows u (float32, oldest first); zeros count for a request without context,
// whatever its slot holds.  Everything is float32 between the load and the store; a token's result does not depend on
// how its request was cut into steps.  A thread walks CV_TOKENS tokens with the window in registers; only the CTAs of a
// request's first tokens read its state, and they write the new one.
#include "common.cuh"
#include <math.h>

#define CV_TOKENS 16           // tokens of a thread (at least taps - 1: the history of later CTAs lies in the step's rows)
#define CV_MAX_TAPS 16
#define CV_THREADS 128

template <typename T, int N> struct CvVec;
template <> struct CvVec<float, 1> { static __device__ __forceinline__ void ld(const float* p, float (&f)[1]) { f[0] = *p; }
                                     static __device__ __forceinline__ void st(float* p, const float (&f)[1]) { *p = f[0]; } };
template <> struct CvVec<float, 2> {
  static __device__ __forceinline__ void ld(const float* p, float (&f)[2]) { const float2 v = *reinterpret_cast<const float2*>(p); f[0] = v.x; f[1] = v.y; }
  static __device__ __forceinline__ void st(float* p, const float (&f)[2]) { *reinterpret_cast<float2*>(p) = make_float2(f[0], f[1]); } };
template <> struct CvVec<__nv_bfloat16, 2> {
  static __device__ __forceinline__ void ld(const __nv_bfloat16* p, float (&f)[2]) {
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); f[0] = a.x; f[1] = a.y; }
  static __device__ __forceinline__ void st(__nv_bfloat16* p, const float (&f)[2]) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(f[0], f[1]); } };
template <> struct CvVec<float, 4> {
  static __device__ __forceinline__ void ld(const float* p, float (&f)[4]) {
    const float4 v = *reinterpret_cast<const float4*>(p); f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w; }
  static __device__ __forceinline__ void st(float* p, const float (&f)[4]) { *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]); } };
template <> struct CvVec<__nv_bfloat16, 1> {
  static __device__ __forceinline__ void ld(const __nv_bfloat16* p, float (&f)[1]) { f[0] = __bfloat162float(*p); }
  static __device__ __forceinline__ void st(__nv_bfloat16* p, const float (&f)[1]) { *p = __float2bfloat16_rn(f[0]); } };
template <> struct CvVec<__nv_bfloat16, 4> {
  static __device__ __forceinline__ void ld(const __nv_bfloat16* p, float (&f)[4]) {
    const uint2 r = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y; }
  static __device__ __forceinline__ void st(__nv_bfloat16* p, const float (&f)[4]) {
    __nv_bfloat162 lo = __floats2bfloat162_rn(f[0], f[1]), hi = __floats2bfloat162_rn(f[2], f[3]);
    uint2 r;
    r.x = *reinterpret_cast<uint32_t*>(&lo); r.y = *reinterpret_cast<uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(p) = r; } };

struct ConvArgs {
  const void* x; long ldx;               // [T, C] in the compute type, rows strided
  const float* in_bias;                  // null, or [C]
  const float* w;                        // [taps, C]; null (taps = 1): y = u
  float* state;                          // [slots, taps - 1, C]
  const int* cu_q; const int* ctx_lens; const int* slot_ids;
  int C, taps, write_state;
};

// A thread's channels c .. c + VEC - 1 of one request: their weights, the window of the last inputs, and the state's move.
// Weights and window are laid out for MT taps whatever the convolution's are: the newest input is last, and taps that the
// convolution does not have weigh nothing.
template <typename T, int VEC, int MT>
struct ConvColumn {
  float w[MT][VEC], win[MT][VEC], bias[VEC];          // (win[MT - 1] is the input that is on its way in)
  const T* x; long ldx; float* st;
  int C, hist;

  // weights: nothing of the step writes them (may run before the wait for the kernel before this one)
  __device__ __forceinline__ void weights(const ConvArgs& A, int c) {
    C = A.C; hist = A.taps - 1;
#pragma unroll
    for (int j = 0; j < MT; ++j) {
      const int tap = j - (MT - 1 - hist);
#pragma unroll
      for (int i = 0; i < VEC; ++i) w[j][i] = (A.w == nullptr && j == MT - 1) ? 1.f : 0.f;
      if (A.w && tap >= 0) CvVec<float, VEC>::ld(A.w + (size_t)tap * C + c, w[j]);
    }
#pragma unroll
    for (int i = 0; i < VEC; ++i) bias[i] = 0.f;
    if (A.in_bias) CvVec<float, VEC>::ld(A.in_bias + c, bias);
  }
  __device__ __forceinline__ void input(int row0, int t, bool has_ctx, float (&u)[VEC]) const {
    if (t >= 0) {
      CvVec<T, VEC>::ld(x + (size_t)(row0 + t) * ldx, u);
#pragma unroll
      for (int i = 0; i < VEC; ++i) u[i] += bias[i];
    } else if (has_ctx && hist + t >= 0) {
      CvVec<float, VEC>::ld(st + (size_t)(hist + t) * C, u);
    } else {
#pragma unroll
      for (int i = 0; i < VEC; ++i) u[i] = 0.f;
    }
  }
  __device__ __forceinline__ void open(const ConvArgs& A, int c, int slot, int row0, int t0, bool has_ctx) {
    x = (const T*)A.x + c; ldx = A.ldx;
    st = A.state ? A.state + (size_t)slot * hist * C + c : nullptr;
#pragma unroll
    for (int j = 0; j < MT - 1; ++j) {
      const int back = MT - 1 - j;                    // tokens before t0
#pragma unroll
      for (int i = 0; i < VEC; ++i) win[j][i] = 0.f;
      if (back <= hist) input(row0, t0 - back, has_ctx, win[j]);
    }
  }
  // y of the input u, which becomes the window's newest
  __device__ __forceinline__ void step(const float (&u)[VEC], float (&y)[VEC]) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      win[MT - 1][i] = u[i];
      float acc = 0.f;
#pragma unroll
      for (int j = 0; j < MT; ++j) acc = fmaf(w[j][i], win[j][i], acc);
      y[i] = acc;
#pragma unroll
      for (int j = 0; j < MT - 1; ++j) win[j][i] = win[j + 1][i];
    }
  }
  // the state's new rows: the last taps - 1 inputs of the request, from the step's rows and, where those are fewer, from
  // the state as it was.  (old rows are read in ascending order ahead of the place they move to)
  __device__ __forceinline__ void close(int row0, int n, bool has_ctx) {
    for (int j = 0; j < hist; ++j) {
      float u[VEC];
      input(row0, n - hist + j, has_ctx, u);
      CvVec<float, VEC>::st(st + (size_t)j * C, u);
    }
  }
};

// ---------------------------------------------------------------------------------------------------------
template <typename T, int VEC, int MT>
__global__ void __launch_bounds__(CV_THREADS, MT == 4 ? 8 : 1)
conv_act_kernel(ConvArgs A, const float* __restrict__ out_bias, T* __restrict__ out, long ldo, int silu) {
  pdl_launch_dependents();
  const int c = (blockIdx.x * CV_THREADS + threadIdx.x) * VEC, req = blockIdx.y, t0 = blockIdx.z * CV_TOKENS;
  const bool in = c < A.C;
  ConvColumn<T, VEC, MT> col;
  float ob[VEC];
#pragma unroll
  for (int i = 0; i < VEC; ++i) ob[i] = 0.f;
  if (in) {
    col.weights(A, c);
    if (out_bias) CvVec<float, VEC>::ld(out_bias + c, ob);
  }
  pdl_wait();
  const int row0 = A.cu_q[req], n = A.cu_q[req + 1] - row0;
  if (!in || t0 >= n) return;
  const bool has_ctx = A.ctx_lens[req] > 0;
  col.open(A, c, A.slot_ids[req], row0, t0, has_ctx);
  const int t1 = min(n, t0 + CV_TOKENS);
  constexpr int AHEAD = 2;                           // inputs on their way at a time (warps hide the latency: more of them beat more loads a thread)
  for (int t = t0; t < t1; t += AHEAD) {
    float u[AHEAD][VEC];
#pragma unroll
    for (int a = 0; a < AHEAD; ++a) if (t + a < t1) col.input(row0, t + a, has_ctx, u[a]);
#pragma unroll
    for (int a = 0; a < AHEAD; ++a) {
      if (t + a >= t1) break;
      float y[VEC];
      col.step(u[a], y);
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        y[i] += ob[i];
        if (silu) y[i] = act_for<T>(y[i], 3);           // (the hardware's exponential and quotient where the result is rounded to bfloat16)
      }
      CvVec<T, VEC>::st(out + (size_t)(row0 + t + a) * ldo + c, y);
    }
  }
  if (t0 == 0 && A.write_state) col.close(row0, n, has_ctx);
}

// ---------------------------------------------------------------------------------------------------------
struct ConvQkvArgs {
  const int* positions; const float* inv_freq; const float2* cos_sin;      // cos_sin null, or [T, rot_dims / 2]
  void* q; long ldq;                                   // [T, H D]
  void* pages; const int* slot_mapping;                // [num_pages, 1 + VP, Hkv, page, D]; null: keys and values are not written
  int H, Hkv, VP, D, rot, page_size;                   // VP: blocks of D value channels per kv head
};

// A thread owns two pieces of VEC channels of one head: the two sides of the pairs that turn together, or two pieces of
// the channels that do not turn.
template <typename T, int VEC, int MT>
__global__ void __launch_bounds__(CV_THREADS, MT == 4 ? 8 : 1)
conv_qkv_kernel(ConvArgs A, ConvQkvArgs Q) {
  pdl_launch_dependents();
  const int D = Q.D, per_head = D / 2 / VEC;
  const int u = blockIdx.x * CV_THREADS + threadIdx.x, req = blockIdx.y, t0 = blockIdx.z * CV_TOKENS;
  const int head = u / per_head, x = (u - head * per_head) * VEC;
  const bool in = head < Q.H + Q.Hkv * (1 + Q.VP);
  const bool is_q = head < Q.H, is_v = head >= Q.H + Q.Hkv;
  const int rot = is_v ? 0 : Q.rot;
  const bool turns = x < rot / 2;
  const int da = turns ? x : rot + (x - rot / 2), db = turns ? x + rot / 2 : rot + (D - rot) / 2 + (x - rot / 2);
  ConvColumn<T, VEC, MT> ca, cb;
  float freq[VEC];
#pragma unroll
  for (int i = 0; i < VEC; ++i) freq[i] = (in && turns) ? Q.inv_freq[x + i] : 0.f;
  if (in) { ca.weights(A, head * D + da); cb.weights(A, head * D + db); }
  pdl_wait();
  const int row0 = A.cu_q[req], n = A.cu_q[req + 1] - row0;
  if (!in || t0 >= n) return;
  const bool has_ctx = A.ctx_lens[req] > 0;
  const int slot = A.slot_ids[req];
  ca.open(A, head * D + da, slot, row0, t0, has_ctx);
  cb.open(A, head * D + db, slot, row0, t0, has_ctx);
  // where the head's rows go: the queries' buffer, or plane (0 keys, 1 + v the v-th block of values) and kv head of a page
  const int vh = head - Q.H - Q.Hkv;
  const int plane = is_v ? 1 + vh % Q.VP : 0, hkv = is_v ? vh / Q.VP : head - Q.H;
  const int t1 = min(n, t0 + CV_TOKENS);
  constexpr int AHEAD = 2;
  for (int t = t0; t < t1; t += AHEAD) {
    float ua[AHEAD][VEC], ub[AHEAD][VEC];
#pragma unroll
    for (int a = 0; a < AHEAD; ++a) if (t + a < t1) { ca.input(row0, t + a, has_ctx, ua[a]); cb.input(row0, t + a, has_ctx, ub[a]); }
#pragma unroll
    for (int a = 0; a < AHEAD; ++a) {
      if (t + a >= t1) break;
      float ya[VEC], yb[VEC];
      ca.step(ua[a], ya);
      cb.step(ub[a], yb);
      const size_t row = (size_t)(row0 + t + a);
      if (turns) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
          float s, c;
          if (Q.cos_sin) { const float2 cs = Q.cos_sin[row * (rot / 2) + x + i]; c = cs.x; s = cs.y; }
          else sincosf((float)Q.positions[row] * freq[i], &s, &c);
          const float p = ya[i], r = yb[i];
          ya[i] = p * c - r * s;
          yb[i] = r * c + p * s;
        }
      }
      T* dst;
      if (is_q) dst = (T*)Q.q + row * Q.ldq + (size_t)head * D;
      else {
        if (Q.pages == nullptr) continue;
        const int sl = Q.slot_mapping[row];
        const int page = sl / Q.page_size, off = sl - page * Q.page_size;
        dst = (T*)Q.pages + ((((size_t)page * (1 + Q.VP) + plane) * Q.Hkv + hkv) * Q.page_size + off) * D;
      }
      CvVec<T, VEC>::st(dst + da, ya);
      CvVec<T, VEC>::st(dst + db, yb);
    }
  }
  if (t0 == 0 && A.write_state) { ca.close(row0, n, has_ctx); cb.close(row0, n, has_ctx); }
}

static int conv_check(const char* name, const ConvArgs& A, int R, int max_q_len) {
  if (A.taps < 1 || A.taps > CV_MAX_TAPS) QE_REFUSE("%s: %d taps are outside 1..%d", name, A.taps, CV_MAX_TAPS);
  if (A.taps > 1 && (A.state == nullptr || A.w == nullptr)) QE_REFUSE("%s: %d taps need weights and a state", name, A.taps);
  if (R > 65535 || (max_q_len + CV_TOKENS - 1) / CV_TOKENS > 65535) QE_REFUSE("%s: %d requests, portions of %d tokens", name, R, max_q_len);
  return 0;
}
static bool conv_aligned(const ConvArgs& A, size_t esize) {
  return A.C % 4 == 0 && A.ldx % 4 == 0 && ((uintptr_t)A.x % (4 * esize)) == 0 && (((uintptr_t)A.in_bias | (uintptr_t)A.w | (uintptr_t)A.state) & 15) == 0;
}

extern "C" int qe_conv_act(const void* x, long ldx, const float* in_bias, const float* w, float* state, const int* cu_q,
                           const int* ctx_lens, const int* slot_ids, const float* out_bias, void* out, long ldo, int R,
                           int max_q_len, int C, int taps, int write_state, int silu, int dtype, cudaStream_t stream) {
  if (R <= 0 || C <= 0 || max_q_len <= 0) return 0;
  ConvArgs A{x, ldx, in_bias, w, state, cu_q, ctx_lens, slot_ids, C, taps, write_state && taps > 1};
  if (int rc = conv_check("conv_act", A, R, max_q_len)) return rc;
  if (dtype != QE_DTYPE_F32 && dtype != QE_DTYPE_BF16) QE_REFUSE("conv_act: unknown dtype %d", dtype);
  const size_t es = dtype == QE_DTYPE_F32 ? 4 : 2;
  const bool vec = conv_aligned(A, es) && ldo % 4 == 0 && ((uintptr_t)out % (4 * es)) == 0 && ((uintptr_t)out_bias & 15) == 0;
  const int V = vec && taps <= 4 ? 4 : 1;
  dim3 grid((unsigned)((C / V + CV_THREADS - 1) / CV_THREADS), R, (max_q_len + CV_TOKENS - 1) / CV_TOKENS);
#define CVA(TT, VV, MM) qe_launch(conv_act_kernel<TT, VV, MM>, grid, dim3(CV_THREADS), 0, stream, A, out_bias, (TT*)out, ldo, silu)
#define CVA_T(TT) do { if (taps > 4) CVA(TT, 1, CV_MAX_TAPS); else if (V == 4) CVA(TT, 4, 4); else CVA(TT, 1, 4); } while (0)
  if (dtype == QE_DTYPE_F32) CVA_T(float); else CVA_T(__nv_bfloat16);
#undef CVA_T
#undef CVA
  QE_CHECK_LAUNCH("conv_act");
  return 0;
}

extern "C" int qe_conv_qkv(const void* x, long ldx, const float* in_bias, const float* w, float* state, const int* cu_q,
                           const int* ctx_lens, const int* slot_ids, const int* positions, const float* inv_freq,
                           const float* cos_sin, int rot_dims, void* q, long ldq, void* pages, const int* slot_mapping, int R,
                           int max_q_len, int H, int Hkv, int value_planes, int D, int page_size, int taps, int write_state,
                           int dtype, cudaStream_t stream) {
  if (R <= 0 || max_q_len <= 0) return 0;
  if (H < 1 || Hkv < 1 || value_planes < 1 || D < 2 || D % 2) QE_REFUSE("conv_qkv: heads %d/%d, %d planes of values, head size %d", H, Hkv, value_planes, D);
  if (rot_dims < 0 || rot_dims > D || rot_dims % 2 || (rot_dims && (inv_freq == nullptr || positions == nullptr)))
    QE_REFUSE("conv_qkv: %d rotated channels of %d", rot_dims, D);
  ConvArgs A{x, ldx, in_bias, w, state, cu_q, ctx_lens, slot_ids, (H + Hkv * (1 + value_planes)) * D, taps, write_state && taps > 1};
  if (int rc = conv_check("conv_qkv", A, R, max_q_len)) return rc;
  if (dtype != QE_DTYPE_F32 && dtype != QE_DTYPE_BF16) QE_REFUSE("conv_qkv: unknown dtype %d", dtype);
  const size_t es = dtype == QE_DTYPE_F32 ? 4 : 2;
  ConvQkvArgs Q{positions, inv_freq, (const float2*)cos_sin, q, ldq, pages, slot_mapping, H, Hkv, value_planes, D, rot_dims, page_size};
  const bool vec = conv_aligned(A, es) && D % 4 == 0 && rot_dims % 4 == 0 && ldq % 4 == 0 && ((uintptr_t)q % (4 * es)) == 0 &&
                   ((uintptr_t)pages % (4 * es)) == 0;
  const int V = vec && taps <= 4 ? 2 : 1;
  const long units = (long)(A.C / 2 / V);
  dim3 grid((unsigned)((units + CV_THREADS - 1) / CV_THREADS), R, (max_q_len + CV_TOKENS - 1) / CV_TOKENS);
#define CVQ(TT, VV, MM) qe_launch(conv_qkv_kernel<TT, VV, MM>, grid, dim3(CV_THREADS), 0, stream, A, Q)
#define CVQ_T(TT) do { if (taps > 4) CVQ(TT, 1, CV_MAX_TAPS); else if (V == 2) CVQ(TT, 2, 4); else CVQ(TT, 1, 4); } while (0)
  if (dtype == QE_DTYPE_F32) CVQ_T(float); else CVQ_T(__nv_bfloat16);
#undef CVQ_T
#undef CVQ
  QE_CHECK_LAUNCH("conv_qkv");
  return 0;
}
