// Recurrences whose state is one matrix per head and whose decay is ONE number per head and token, as a scan over the
// tokens of every request, state in float32:
//
//   S_t = a_t S_(t-1) + b_t k_t v_t^T      (S: dk key channels x dv value channels)
//   o_t = S_t^T (q_scale q_t) (+ skip_h v_t)
//
// Two ways to get a and b from what a projection returned for the token (float32 arithmetic):
//   form 0, a state-space model: dt = softplus(g0 + b0_h), a = exp(-exp(log_rate_h) dt), b = dt;
//   form 1, a matrix memory with exponential gates: i = cap tanh((g0 + b0_h) / cap), f = logsigmoid(cap tanh((g1 + b1_h) / cap)),
//           m_t = max(f + m_(t-1), i) from m = 0, a = exp(f + m_(t-1) - m_t), b = exp(i - m_t).  The memory then has one value
//           channel more, whose value is 1 for every token: its column is the normaliser n, and den[t, h] =
//           max(|n_t . q_t|, exp(-m_t)) + den_eps is what the head's output is to be divided by.
// q, k [T, G dk] (head h reads group h / (H / G)) and v [T, H dv] come in the compute type.
//
// The scan: one CTA per (request, head, tile of value channels).  A value channel's column of S evolves on its own; a
// thread owns J columns x DC consecutive key channels in registers, so that a staged q and k serve J columns; the L
// threads of a column group are neighbours in one warp.  Every multiply-add works on a pair of channels.  Four producer
// warps stage the next chunk of tokens in shared memory as float32; the first of them also forms the chunk's a and b (for
// form 1 it carries m).  Four tokens a turn: their J sums each are exchanged together (a lane ends up with its share).
// The order of every sum depends on the sizes alone, so a token's output does not depend on how its request was cut.
//
// Steps of single tokens take a kernel of their own: nothing is staged, a thread's part of the state is on its way before
// the kernel waits for the one before it.
//
// State: [slot][head][dv (+ 1)][dk] float32, and for form 1 m in [slot][head][dv + 1] (each column's CTA keeps the copies
// of its columns, so that no CTA reads what another writes).  A request without context starts from zero.
#include "common.cuh"
#include <math.h>

#define MS_COMPUTE 128
#define MS_PRODUCERS 128
#define MS_SMEM_MAX (110 * 1024)

struct MsArgs {
  const void* q; const void* k; const void* v; long ldq, ldk, ldv;
  float* state; float* mstate;
  const int* cu_q; const int* ctx_lens; const int* slot_ids;
  float* out; float* den;                               // [T, H dv]; form 1: [T, H]
  const void* g0; const void* g1; long ldg0, ldg1; int gates_f32;     // [T, H]: compute type, or float32
  const float* b0; const float* b1; const float* log_rate; const float* skip;
  float cap, q_scale, den_eps;
  int form, H, G, dk, dv, dvx, VT, chunk, write_state, vec;
};

__device__ __forceinline__ float2 ms_fma2(float2 a, float2 b, float2 c) {
  float2 d;
  asm("{\n\t.reg .b64 ra, rb, rc, rd;\n\t"
      "mov.b64 ra, {%2, %3};\n\tmov.b64 rb, {%4, %5};\n\tmov.b64 rc, {%6, %7};\n\t"
      "fma.rn.f32x2 rd, ra, rb, rc;\n\t"
      "mov.b64 {%0, %1}, rd;\n\t}\n"
      : "=f"(d.x), "=f"(d.y) : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y), "f"(c.x), "f"(c.y));
  return d;
}
__device__ __forceinline__ float2 ms_mul2(float2 a, float2 b) {
  float2 d;
  asm("{\n\t.reg .b64 ra, rb, rd;\n\t"
      "mov.b64 ra, {%2, %3};\n\tmov.b64 rb, {%4, %5};\n\t"
      "mul.rn.f32x2 rd, ra, rb;\n\t"
      "mov.b64 {%0, %1}, rd;\n\t}\n"
      : "=f"(d.x), "=f"(d.y) : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y));
  return d;
}

template <typename T>
__device__ __forceinline__ float ms_gate_in(const void* g, long ld, int f32, size_t row, int head) {
  return f32 ? ((const float*)g)[row * ld + head] : to_f32(((const T*)g)[row * ld + head]);
}
// form 1's log gates
__device__ __forceinline__ float ms_log_in(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float ms_log_keep(float z, float cap) {
  const float s = cap * tanhf(z / cap);
  return fminf(s, 0.f) - log1pf(expf(-fabsf(s)));
}
// form 0's step
__device__ __forceinline__ float ms_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// one token on a thread's J columns of DC channels: the state moves on, acc = q . s
template <int DC, int J>
__device__ __forceinline__ void ms_token(float2 (&s)[J][DC / 2], const float* qr, const float* kr, const float (&u)[J], float a,
                                         float (&acc)[J]) {
  float2 sum[J];
#pragma unroll
  for (int j = 0; j < J; ++j) sum[j] = make_float2(0.f, 0.f);
  const float2 a2 = make_float2(a, a);
#pragma unroll
  for (int i = 0; i < DC; i += 4) {
    const float4 q4 = *reinterpret_cast<const float4*>(qr + i);
    const float4 k4 = *reinterpret_cast<const float4*>(kr + i);
#pragma unroll
    for (int j = 0; j < J; ++j) {
      const float2 u2 = make_float2(u[j], u[j]);
      float2& s0 = s[j][i / 2];
      float2& s1 = s[j][i / 2 + 1];
      s0 = ms_fma2(a2, s0, ms_mul2(make_float2(k4.x, k4.y), u2));
      s1 = ms_fma2(a2, s1, ms_mul2(make_float2(k4.z, k4.w), u2));
      sum[j] = ms_fma2(make_float2(q4.x, q4.y), s0, sum[j]);
      sum[j] = ms_fma2(make_float2(q4.z, q4.w), s1, sum[j]);
    }
  }
#pragma unroll
  for (int j = 0; j < J; ++j) acc[j] = sum[j].x + sum[j].y;
}

template <int DC, int J>
__device__ __forceinline__ void ms_load_state(float2 (&s)[J][DC / 2], const float* st, int dk, int l, int j_first, int j_end, bool has) {
#pragma unroll
  for (int j = 0; j < J; ++j) {
#pragma unroll
    for (int i = 0; i < DC / 2; ++i) s[j][i] = make_float2(0.f, 0.f);
    if (!has || j_first + j >= j_end) continue;
    const float* r = st + (size_t)(j_first + j) * dk;
    if (dk % 4 == 0) {
#pragma unroll
      for (int i = 0; i < DC; i += 4) {
        const int c = l * DC + i;
        if (c < dk) {
          const float4 x = *reinterpret_cast<const float4*>(r + c);
          s[j][i / 2] = make_float2(x.x, x.y); s[j][i / 2 + 1] = make_float2(x.z, x.w);
        }
      }
    } else {
#pragma unroll
      for (int i = 0; i < DC; i += 2) {
        const int c = l * DC + i;
        if (c < dk) s[j][i / 2].x = r[c];
        if (c + 1 < dk) s[j][i / 2].y = r[c + 1];
      }
    }
  }
}
template <int DC, int J>
__device__ __forceinline__ void ms_store_state(const float2 (&s)[J][DC / 2], float* st, int dk, int l, int j_first, int j_end) {
#pragma unroll
  for (int j = 0; j < J; ++j) {
    if (j_first + j >= j_end) continue;
    float* r = st + (size_t)(j_first + j) * dk;
    if (dk % 4 == 0) {
#pragma unroll
      for (int i = 0; i < DC; i += 4) {
        const int c = l * DC + i;
        if (c < dk) *reinterpret_cast<float4*>(r + c) = make_float4(s[j][i / 2].x, s[j][i / 2].y, s[j][i / 2 + 1].x, s[j][i / 2 + 1].y);
      }
    } else {
#pragma unroll
      for (int i = 0; i < DC; i += 2) {
        const int c = l * DC + i;
        if (c < dk) r[c] = s[j][i / 2].x;
        if (c + 1 < dk) r[c + 1] = s[j][i / 2].y;
      }
    }
  }
}

// index of key channel c in a staged row: blocks of DC channels with 4 floats between them (banks)
template <int DC> __device__ __forceinline__ int ms_pad(int c) { return c + (c / DC) * 4; }

template <typename T, int DC, int J, int L>
__global__ void __launch_bounds__(MS_COMPUTE + MS_PRODUCERS)
memory_scan_kernel(MsArgs A) {
  extern __shared__ __align__(16) float smem[];
  const int req = blockIdx.x, head = blockIdx.y, VT = A.VT, j0 = blockIdx.z * VT;
  const int dk = A.dk, dv = A.dv, dvx = A.dvx, H = A.H;
  constexpr int row_w = L * (DC + 4);
  const int VTp = (VT + 3) & ~3;
  const int tok_w = 2 * row_w + VTp + 4;                // q, k, v of the tile, (a, b, exp(-m))
  auto buf = [&](int ch) { return smem + (size_t)(ch & 1) * A.chunk * tok_w; };
  const int n_compute = blockDim.x - MS_PRODUCERS;
  const int tid = threadIdx.x;
  const bool producer = tid >= n_compute;
  const int l = tid % L, cg = tid / L;
  const int jc = j0 + cg * J;                           // the thread's first column
  const int j_end = min(dvx, j0 + VT);
  pdl_launch_dependents();
  const int row0 = A.cu_q[req];                         // (the step's index data: the host's copy)
  const int n = A.cu_q[req + 1] - row0;
  const int ctx = A.ctx_lens[req], slot = A.slot_ids[req];
  if (n <= 0) { pdl_wait(); return; }
  const int n_chunks = (n + A.chunk - 1) / A.chunk;
  const int chunk = A.chunk;
  float* st = A.state + ((size_t)slot * H + head) * dvx * dk;
  float* ms = A.mstate ? A.mstate + ((size_t)slot * H + head) * dvx : nullptr;

  if (producer) {
    const int ptid = tid - n_compute, plane_ = tid & 31;
    const int grp = head / (H / A.G);
    const T* q = (const T*)A.q + (size_t)grp * dk;
    const T* k = (const T*)A.k + (size_t)grp * dk;
    const T* v = (const T*)A.v + (size_t)head * dv;
    const float bias0 = A.b0 ? A.b0[head] : 0.f, bias1 = A.b1 ? A.b1[head] : 0.f;
    const float rate = A.log_rate ? expf(A.log_rate[head]) : 0.f;
    float m = (A.form == 1 && ctx > 0) ? ms[j0] : 0.f;
    // what no copy writes: key channels beyond the head, in both buffers
    if (L * DC > dk)
      for (int e = ptid; e < 2 * chunk * (L * DC - dk); e += MS_PRODUCERS) {
        const int t = e / (L * DC - dk), c = dk + e - t * (L * DC - dk);
        float* dst = smem + (size_t)t * tok_w + ms_pad<DC>(c);
        dst[0] = 0.f; dst[row_w] = 0.f;
      }
    pdl_wait();
    constexpr int VEC = 16 / (int)sizeof(T);
    auto stage = [&](int ch) {
      float* b = buf(ch);
      const int t_first = ch * chunk, rows = min(chunk, n - t_first), rows4 = min((rows + 3) & ~3, chunk);
      // a and b of the chunk's tokens: one warp, a token a lane (32 at most a turn)
      if (ptid < 32) {
        for (int tb = 0; tb < rows4; tb += 32) {
          const int t = tb + plane_;
          float a = 1.f, bb = 0.f, fl = 0.f;
          const size_t row = (size_t)(row0 + t_first + t);
          if (A.form == 0) {
            if (t < rows) {
              const float dt = ms_softplus(ms_gate_in<T>(A.g0, A.ldg0, A.gates_f32, row, head) + bias0);
              a = expf(-rate * dt); bb = dt;
            }
          } else {
            float gi = 0.f, gf = 0.f;
            if (t < rows) {
              gi = ms_log_in(ms_gate_in<T>(A.g0, A.ldg0, A.gates_f32, row, head) + bias0, A.cap);
              gf = ms_log_keep(ms_gate_in<T>(A.g1, A.ldg1, A.gates_f32, row, head) + bias1, A.cap);
            }
            float kept = 0.f, mine = 0.f;
            const int n_here = min(32, rows - tb);
            for (int x = 0; x < n_here; ++x) {
              const float fx = __shfl_sync(0xffffffffu, gf, x), ix = __shfl_sync(0xffffffffu, gi, x);
              const float kx = fx + m;
              m = fmaxf(kx, ix);
              if (x == plane_) { kept = kx; mine = m; }
            }
            if (t < rows) { a = expf(kept - mine); bb = expf(gi - mine); fl = expf(-mine); }
          }
          if (t < rows4) *reinterpret_cast<float4*>(b + (size_t)t * tok_w + 2 * row_w + VTp) = make_float4(a, bb, fl, 0.f);
        }
      }
      if (A.vec) {
        // pieces of 16 bytes: q, k of the group, v of the tile; several loads on their way before the first is stored
        const int pk = dk / VEC, pv = VT / VEC, per = 2 * pk + pv;
        const int total = rows * per;
        constexpr int NI = 4;
        for (int e0 = ptid; e0 < total; e0 += NI * MS_PRODUCERS) {
          uint4 r[NI];
          int dst[NI], kind[NI];
#pragma unroll
          for (int i = 0; i < NI; ++i) {
            const int e = e0 + i * MS_PRODUCERS;
            kind[i] = -1;
            if (e >= total) continue;
            const int t = e / per;
            int x = e - t * per;
            const size_t row = (size_t)(row0 + t_first + t);
            const T* src;
            if (x < pk) { kind[i] = 0; src = q + row * A.ldq + x * VEC; dst[i] = t * tok_w + ms_pad<DC>(x * VEC); }
            else if ((x -= pk) < pk) { kind[i] = 1; src = k + row * A.ldk + x * VEC; dst[i] = t * tok_w + row_w + ms_pad<DC>(x * VEC); }
            else {
              x -= pk;
              kind[i] = 2; dst[i] = t * tok_w + 2 * row_w + x * VEC;
              src = v + row * A.ldv + j0 + x * VEC;
              if (j0 + x * VEC >= dv) { kind[i] = j0 + x * VEC == dv ? 3 : 4; continue; }     // the normaliser's column, or beyond
            }
            r[i] = __ldg(reinterpret_cast<const uint4*>(src));
          }
#pragma unroll
          for (int i = 0; i < NI; ++i) {
            if (kind[i] < 0) continue;
            float f[VEC];
            if (kind[i] >= 3) {
#pragma unroll
              for (int x = 0; x < VEC; ++x) f[x] = (kind[i] == 3 && x == 0) ? 1.f : 0.f;
            } else if constexpr (sizeof(T) == 2) {
              const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&r[i]);
#pragma unroll
              for (int x = 0; x < 4; ++x) { const float2 y = __bfloat1622float2(h2[x]); f[2 * x] = y.x; f[2 * x + 1] = y.y; }
            } else {
              f[0] = __uint_as_float(r[i].x); f[1] = __uint_as_float(r[i].y); f[2] = __uint_as_float(r[i].z); f[3] = __uint_as_float(r[i].w);
            }
            if (kind[i] == 0) {
#pragma unroll
              for (int x = 0; x < VEC; ++x) f[x] *= A.q_scale;
            }
            // (a piece lies within one block of DC channels: DC is a multiple of VEC)
            *reinterpret_cast<float4*>(b + dst[i]) = make_float4(f[0], f[1], f[2], f[3]);
            if constexpr (VEC == 8) *reinterpret_cast<float4*>(b + dst[i] + 4) = make_float4(f[4], f[5], f[6], f[7]);
          }
        }
      } else {
        const int per = 2 * dk + VT;
        for (int e = ptid; e < rows * per; e += MS_PRODUCERS) {
          const int t = e / per;
          int x = e - t * per;
          const size_t row = (size_t)(row0 + t_first + t);
          float* dst = b + (size_t)t * tok_w;
          if (x < dk) dst[ms_pad<DC>(x)] = to_f32(q[row * A.ldq + x]) * A.q_scale;
          else if ((x -= dk) < dk) dst[row_w + ms_pad<DC>(x)] = to_f32(k[row * A.ldk + x]);
          else {
            x -= dk;
            dst[2 * row_w + x] = j0 + x < dv ? to_f32(v[row * A.ldv + j0 + x]) : (j0 + x == dv ? 1.f : 0.f);
          }
        }
      }
      // tokens that fill the last turn of four: nothing in, nothing decays (their outputs are not stored)
      for (int e = ptid; e < (rows4 - rows) * (2 * row_w + VTp); e += MS_PRODUCERS) {
        const int t = e / (2 * row_w + VTp), x = e - t * (2 * row_w + VTp);
        b[(size_t)(rows + t) * tok_w + x] = 0.f;
      }
    };
    stage(0);
    __syncthreads();
    for (int ch = 0; ch < n_chunks; ++ch) {
      if (ch + 1 < n_chunks) stage(ch + 1);
      __syncthreads();
    }
    if (A.form == 1 && A.write_state && ptid < 32)
      for (int j = j0 + plane_; j < j_end; j += 32) ms[j] = m;
    return;
  }

  // ---- the columns ----------------------------------------------------------------------------------------
  float2 s[J][DC / 2];
  ms_load_state<DC, J>(s, st, dk, l, jc, j_end, ctx > 0);
  float skip = A.skip ? A.skip[head] : 0.f;
  pdl_wait();
  __syncthreads();
  const size_t o_ld = (size_t)H * dv;
  for (int ch = 0; ch < n_chunks; ++ch) {
    const int rows = min(chunk, n - ch * chunk);
    const float* r = buf(ch);
    const size_t row = (size_t)(row0 + ch * chunk);
    for (int t0 = 0; t0 < rows; t0 += 4, r += 4 * tok_w) {
      constexpr int NV = 4 * J;
      float val[NV];                                    // [token][column]
#pragma unroll
      for (int t = 0; t < 4; ++t) {
        const float* rt = r + t * tok_w;
        const float2 ab = *reinterpret_cast<const float2*>(rt + 2 * row_w + VTp);
        float u[J], acc[J];
#pragma unroll
        for (int j = 0; j < J; ++j) u[j] = ab.y * rt[2 * row_w + cg * J + j];
        ms_token<DC, J>(s, rt + l * (DC + 4), rt + row_w + l * (DC + 4), u, ab.x, acc);
#pragma unroll
        for (int j = 0; j < J; ++j) val[t * J + j] = acc[j];
      }
      // the sums over the column's L lanes: in each round a lane keeps half of its values and hands over the other half
      int mine = 0, held = NV;
#pragma unroll
      for (int off = 1; off < L; off <<= 1) {
        if (held > 1) {
          const bool up = l & off;
          const int half = held / 2;
#pragma unroll
          for (int i = 0; i < NV / 2; ++i) {
            if (i >= half) continue;
            const float give = up ? val[i] : val[i + half], keep = up ? val[i + half] : val[i];
            val[i] = keep + __shfl_xor_sync(0xffffffffu, give, off);
          }
          mine += up ? half : 0;
          held = half;
        } else {
          val[0] += __shfl_xor_sync(0xffffffffu, val[0], off);
        }
      }
      if (L <= NV || l < NV) {
#pragma unroll
        for (int i = 0; i < NV; ++i) {
          if (i >= held) continue;
          const int x = mine + i, t = x / J, j = x - t * J, col = jc + j;
          if (t0 + t >= rows || col >= j_end) continue;
          const float* rt = r + t * tok_w;
          if (col < dv) A.out[(row + t0 + t) * o_ld + (size_t)head * dv + col] = fmaf(skip, rt[2 * row_w + cg * J + j], val[i]);
          else A.den[(row + t0 + t) * H + head] = fmaxf(fabsf(val[i]), rt[2 * row_w + VTp + 2]) + A.den_eps;
        }
      }
    }
    __syncthreads();
  }
  if (A.write_state) ms_store_state<DC, J>(s, st, dk, l, jc, j_end);
}

// A step of single tokens: one token a request.
template <typename T, int DC, int J, int L>
__global__ void __launch_bounds__(MS_COMPUTE)
memory_step_kernel(MsArgs A) {
  const int req = blockIdx.x, head = blockIdx.y, j0 = blockIdx.z * A.VT;
  const int dk = A.dk, dv = A.dv, dvx = A.dvx, H = A.H;
  const int l = threadIdx.x % L, cg = threadIdx.x / L;
  const int jc = j0 + cg * J, j_end = min(dvx, j0 + A.VT);
  pdl_launch_dependents();
  const int row0 = A.cu_q[req], n = A.cu_q[req + 1] - row0;
  const int ctx = A.ctx_lens[req], slot = A.slot_ids[req];
  float* st = A.state + ((size_t)slot * H + head) * dvx * dk;
  float* ms = A.mstate ? A.mstate + ((size_t)slot * H + head) * dvx : nullptr;
  // the state was written by an earlier step: it need not wait for the kernel before this one
  float2 s[J][DC / 2];
  ms_load_state<DC, J>(s, st, dk, l, jc, j_end, ctx > 0 && n > 0);
  const float m_old = (A.form == 1 && ctx > 0) ? ms[j0] : 0.f;
  const float bias0 = A.b0 ? A.b0[head] : 0.f, bias1 = A.b1 ? A.b1[head] : 0.f;
  const float rate = A.log_rate ? expf(A.log_rate[head]) : 0.f, skip = A.skip ? A.skip[head] : 0.f;
  pdl_wait();
  if (n <= 0) return;
  const size_t row = (size_t)row0;
  const int grp = head / (H / A.G);
  const T* q = (const T*)A.q + row * A.ldq + (size_t)grp * dk;
  const T* k = (const T*)A.k + row * A.ldk + (size_t)grp * dk;
  const T* v = (const T*)A.v + row * A.ldv + (size_t)head * dv;
  float qf[DC], kf[DC];
#pragma unroll
  for (int i = 0; i < DC; ++i) {
    const int c = l * DC + i;
    qf[i] = c < dk ? to_f32(q[c]) * A.q_scale : 0.f;
    kf[i] = c < dk ? to_f32(k[c]) : 0.f;
  }
  float vf[J];
#pragma unroll
  for (int j = 0; j < J; ++j) vf[j] = jc + j < dv ? to_f32(v[jc + j]) : (jc + j == dv ? 1.f : 0.f);
  float a, b, fl = 0.f, m = 0.f;
  if (A.form == 0) {
    b = ms_softplus(ms_gate_in<T>(A.g0, A.ldg0, A.gates_f32, row, head) + bias0);
    a = expf(-rate * b);
  } else {
    const float gi = ms_log_in(ms_gate_in<T>(A.g0, A.ldg0, A.gates_f32, row, head) + bias0, A.cap);
    const float kept = ms_log_keep(ms_gate_in<T>(A.g1, A.ldg1, A.gates_f32, row, head) + bias1, A.cap) + m_old;
    m = fmaxf(kept, gi);
    a = expf(kept - m); b = expf(gi - m); fl = expf(-m);
  }
  float u[J], acc[J];
#pragma unroll
  for (int j = 0; j < J; ++j) u[j] = b * vf[j];
  ms_token<DC, J>(s, qf, kf, u, a, acc);
#pragma unroll
  for (int off = 1; off < L; off <<= 1)
#pragma unroll
    for (int j = 0; j < J; ++j) acc[j] += __shfl_xor_sync(0xffffffffu, acc[j], off);
  if (l == 0) {
#pragma unroll
    for (int j = 0; j < J; ++j) {
      const int col = jc + j;
      if (col >= j_end) continue;
      if (col < dv) A.out[row * ((size_t)H * dv) + (size_t)head * dv + col] = fmaf(skip, vf[j], acc[j]);
      else A.den[row * H + head] = fmaxf(fabsf(acc[j]), fl) + A.den_eps;
    }
  }
  if (A.write_state) {
    ms_store_state<DC, J>(s, st, dk, l, jc, j_end);
    // (every thread of the CTA has read its m; the CTA's columns are its own)
    if (A.form == 1) { __syncthreads(); for (int j = j0 + threadIdx.x; j < j_end; j += blockDim.x) ms[j] = m; }
  }
}

// The columns of a CTA: as many as MS_COMPUTE threads hold, fewer where the grid would leave SMs idle.
static int ms_threads(long units, int dvx, int L, int J) {
  int threads = MS_COMPUTE;
  auto tiles = [&](int th) { const int vt = th / L * J; return (long)((dvx + vt - 1) / vt); };
  while (threads > 32 && threads / 2 / L * J >= 8 && (units * tiles(threads) < 148 || threads / 2 / L * J >= dvx)) threads /= 2;
  return threads;
}

template <typename T, int DC, int J, int L>
static int ms_launch(MsArgs A, int R, int max_q_len, cudaStream_t stream) {
  const int threads = ms_threads((long)R * A.H, A.dvx, L, J);
  A.VT = threads / L * J;
  const dim3 grid(R, A.H, (A.dvx + A.VT - 1) / A.VT);
  if (grid.z > 65535) QE_REFUSE("memory_scan: %d value channels are too many", A.dv);
  if (max_q_len <= 1) {
    qe_launch(memory_step_kernel<T, DC, J, L>, grid, dim3(threads), 0, stream, A);
    QE_CHECK_LAUNCH("memory_scan");
    return 0;
  }
  const int tok_w = 2 * L * (DC + 4) + ((A.VT + 3) & ~3) + 4;
  int chunk = 32;
  while (chunk > 4 && ((size_t)2 * chunk * tok_w * 4 > MS_SMEM_MAX || chunk / 2 >= max_q_len)) chunk >>= 1;
  const size_t smem = (size_t)2 * chunk * tok_w * 4;
  if (smem > MS_SMEM_MAX) QE_REFUSE("memory_scan: key size %d needs %zu bytes of shared memory", A.dk, smem);
  A.chunk = chunk;
  const int VEC = 16 / (int)sizeof(T);
  A.vec = A.dk % VEC == 0 && A.dv % VEC == 0 && A.VT % VEC == 0 && A.ldq % VEC == 0 && A.ldk % VEC == 0 && A.ldv % VEC == 0 &&
          (((uintptr_t)A.q | (uintptr_t)A.k | (uintptr_t)A.v) & 15) == 0;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(memory_scan_kernel<T, DC, J, L>, cudaFuncAttributeMaxDynamicSharedMemorySize, MS_SMEM_MAX);
    if (e != cudaSuccess) QE_REFUSE("memory_scan: shared memory: %s", cudaGetErrorString(e));
    configured = true;
  }
  qe_launch(memory_scan_kernel<T, DC, J, L>, grid, dim3(threads + MS_PRODUCERS), smem, stream, A);
  QE_CHECK_LAUNCH("memory_scan");
  return 0;
}

// form 0: gates0 = dt [T, H], bias0 = its bias, log_rate, skip (may be null).  form 1: gates0 and gates1 = the input and
// forget gates [T, H] with their biases, cap, mstate, den and den_eps.  gates_f32: the gates come in float32.
extern "C" int qe_memory_scan(const void* q, long ldq, const void* k, long ldk, const void* v, long ldv, float* state, float* mstate,
                              const int* cu_q, const int* ctx_lens, const int* slot_ids, float* out, float* den, const void* gates0,
                              long ldg0, const void* gates1, long ldg1, int gates_f32, const float* bias0, const float* bias1,
                              const float* log_rate, const float* skip, float cap, float q_scale, float den_eps, int form, int R,
                              int max_q_len, int H, int G, int dk, int dv, int write_state, int dtype, cudaStream_t stream) {
  if (R <= 0 || max_q_len <= 0) return 0;
  if (form != 0 && form != 1) QE_REFUSE("memory_scan: unknown form %d", form);
  if (dk < 1 || dk > 1024 || dv < 1) QE_REFUSE("memory_scan: key size %d must be 1..1024, value size %d positive", dk, dv);
  if (H < 1 || H > 65535 || G < 1 || H % G) QE_REFUSE("memory_scan: %d heads over %d groups", H, G);
  if (gates0 == nullptr || (form == 0 && log_rate == nullptr)) QE_REFUSE("memory_scan: the gates' inputs are missing");
  if (form == 1 && (gates1 == nullptr || mstate == nullptr || den == nullptr || !(cap > 0.f))) QE_REFUSE("memory_scan: form 1 needs both gates, a cap, the maxima and the divisors");
  MsArgs A{q, k, v, ldq, ldk, ldv, state, form == 1 ? mstate : nullptr, cu_q, ctx_lens, slot_ids, out, den, gates0, gates1, ldg0, ldg1,
           gates_f32, bias0, bias1, form == 0 ? log_rate : nullptr, form == 0 ? skip : nullptr, cap, q_scale, den_eps,
           form, H, G, dk, dv, form == 1 ? dv + 1 : dv, 0, 0, write_state, 0};
  int L = 1;
  const int DC = dk <= 256 ? 8 : 32;
  while (L * DC < dk) L <<= 1;
#define MSL(TT) do { \
    if (DC == 8) switch (L) { \
      case 1: return ms_launch<TT, 8, 4, 1>(A, R, max_q_len, stream); case 2: return ms_launch<TT, 8, 4, 2>(A, R, max_q_len, stream); \
      case 4: return ms_launch<TT, 8, 4, 4>(A, R, max_q_len, stream); case 8: return ms_launch<TT, 8, 4, 8>(A, R, max_q_len, stream); \
      case 16: return ms_launch<TT, 8, 4, 16>(A, R, max_q_len, stream); default: return ms_launch<TT, 8, 4, 32>(A, R, max_q_len, stream); } \
    else switch (L) { case 16: return ms_launch<TT, 32, 1, 16>(A, R, max_q_len, stream); default: return ms_launch<TT, 32, 1, 32>(A, R, max_q_len, stream); } \
  } while (0)
  if (dtype == QE_DTYPE_F32) MSL(float);
  else if (dtype == QE_DTYPE_BF16) MSL(__nv_bfloat16);
#undef MSL
  QE_REFUSE("memory_scan: unknown dtype %d", dtype);
}
