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
// threads of a column group are neighbours in one warp.  Every multiply-add works on a pair of channels.  Chunks of tokens
// come through a ring in shared memory (16-byte asynchronous copies, as they are stored); one more warp forms the next
// chunk's a and b (for form 1 it carries m).  A few tokens a turn: their J sums each are exchanged together (a lane ends up
// with its share).  The order of every sum depends on the sizes alone, so a token's output does not depend on how its request was cut.
//
// Steps of single tokens take a kernel of their own: nothing is staged, a thread's part of the state is on its way before
// the kernel waits for the one before it.
//
// State: [slot][head][dv (+ 1)][dk] float32, and for form 1 m in [slot][head][dv + 1] (each column's CTA keeps the copies
// of its columns, so that no CTA reads what another writes).  A request without context starts from zero.
#include "common.cuh"
#include <math.h>

#define MS_STAGES 3                // chunks of tokens in shared memory
#define MS_SMEM_MAX (110 * 1024)
__host__ __device__ constexpr int ms_threads_max(int J) { return J == 2 ? 256 : 128; }   // threads that hold state, at most
__host__ __device__ constexpr int ms_turn(int J) { return J == 4 ? 4 : 8; }      // tokens whose sums are exchanged together

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
__device__ __forceinline__ void ms_token(float2 (&s)[J][DC / 2], const float2 (&q)[DC / 2], const float2 (&k)[DC / 2], const float (&u)[J],
                                         float a, float (&acc)[J]) {
  float2 sum[J];
#pragma unroll
  for (int j = 0; j < J; ++j) sum[j] = make_float2(0.f, 0.f);
  const float2 a2 = make_float2(a, a);
#pragma unroll
  for (int i = 0; i < DC / 2; ++i) {
#pragma unroll
    for (int j = 0; j < J; ++j) {
      s[j][i] = ms_fma2(a2, s[j][i], ms_mul2(k[i], make_float2(u[j], u[j])));
      sum[j] = ms_fma2(q[i], s[j][i], sum[j]);
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

// DC consecutive elements of the compute type in shared memory as pairs of floats
template <int DC> __device__ __forceinline__ void ms_pairs(const __nv_bfloat16* p, float2 (&f)[DC / 2]) {
#pragma unroll
  for (int i = 0; i < DC / 8; ++i) {
    const uint4 r = *reinterpret_cast<const uint4*>(p + 8 * i);
    const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
    for (int x = 0; x < 4; ++x) f[4 * i + x] = make_float2(__uint_as_float(w[x] << 16), __uint_as_float(w[x] & 0xffff0000u));
  }
}
template <int DC> __device__ __forceinline__ void ms_pairs(const float* p, float2 (&f)[DC / 2]) {
#pragma unroll
  for (int i = 0; i < DC / 4; ++i) {
    const float4 r = *reinterpret_cast<const float4*>(p + 4 * i);
    f[2 * i] = make_float2(r.x, r.y); f[2 * i + 1] = make_float2(r.z, r.w);
  }
}
template <int J> __device__ __forceinline__ void ms_values(const __nv_bfloat16* p, float (&v)[J]) {
  if constexpr (J == 4) {
    const uint2 r = *reinterpret_cast<const uint2*>(p);
    v[0] = __uint_as_float(r.x << 16); v[1] = __uint_as_float(r.x & 0xffff0000u);
    v[2] = __uint_as_float(r.y << 16); v[3] = __uint_as_float(r.y & 0xffff0000u);
  } else if constexpr (J == 2) {
    const uint32_t r = *reinterpret_cast<const uint32_t*>(p);
    v[0] = __uint_as_float(r << 16); v[1] = __uint_as_float(r & 0xffff0000u);
  } else v[0] = __bfloat162float(p[0]);
}
template <int J> __device__ __forceinline__ void ms_values(const float* p, float (&v)[J]) {
  if constexpr (J == 4) { const float4 r = *reinterpret_cast<const float4*>(p); v[0] = r.x; v[1] = r.y; v[2] = r.z; v[3] = r.w; }
  else if constexpr (J == 2) { const float2 r = *reinterpret_cast<const float2*>(p); v[0] = r.x; v[1] = r.y; }
  else v[0] = p[0];
}
// 16 bytes to shared memory; not valid: nothing is read and zeros are written
__device__ __forceinline__ void ms_cp_async16(void* smem, const void* gmem, bool valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" :: "r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem), "r"(valid ? 16 : 0));
}

template <typename T, int DC, int J, int L>
__global__ void __launch_bounds__(ms_threads_max(J) + 32, 1)
memory_scan_kernel(MsArgs A) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const int req = blockIdx.x, head = blockIdx.y, VT = A.VT, j0 = blockIdx.z * VT;
  const int dk = A.dk, dv = A.dv, dvx = A.dvx, H = A.H, chunk = A.chunk;
  constexpr int QW = L * DC;                            // elements of a staged row of q or k
  constexpr int VEC = 16 / (int)sizeof(T);
  constexpr int TURN = ms_turn(J);
  const int VTp = (VT + VEC - 1) / VEC * VEC;
  const int stage_elems = chunk * (2 * QW + VTp);       // q rows, k rows, v rows
  T* const stages = reinterpret_cast<T*>(smem_raw);
  float4* const scalars = reinterpret_cast<float4*>(stages + (size_t)MS_STAGES * stage_elems);       // [2][chunk]: a, b, exp(-m)
  const int n_compute = blockDim.x - 32;
  const int tid = threadIdx.x, lane = tid & 31;
  const bool scalar_warp = tid >= n_compute;
  const int l = tid % L, cg = tid / L;
  const int jc = j0 + cg * J;                           // the thread's first column
  const int j_end = min(dvx, j0 + VT);
  pdl_launch_dependents();
  const int row0 = A.cu_q[req];                         // (the step's index data: the host's copy)
  const int n = A.cu_q[req + 1] - row0;
  const int ctx = A.ctx_lens[req], slot = A.slot_ids[req];
  if (n <= 0) { pdl_wait(); return; }
  const int n_chunks = (n + chunk - 1) / chunk;
  float* st = A.state + ((size_t)slot * H + head) * dvx * dk;
  float* ms = A.mstate ? A.mstate + ((size_t)slot * H + head) * dvx : nullptr;

  if (scalar_warp) {
    // ---- a and b of a chunk's tokens, a token a lane; form 1 carries m through them one after the other ----------
    const float bias0 = A.b0 ? A.b0[head] : 0.f, bias1 = A.b1 ? A.b1[head] : 0.f;
    const float rate = A.log_rate ? expf(A.log_rate[head]) : 0.f;
    float m = (A.form == 1 && ctx > 0) ? ms[j0] : 0.f;
    pdl_wait();
    auto form_chunk = [&](int ch) {
      const int t_first = ch * chunk, rows = min(chunk, n - t_first);
      for (int tb = 0; tb < chunk; tb += 32) {
        const int t = tb + lane;
        float a = 1.f, bb = 0.f, fl = 0.f;              // (tokens behind the last: nothing decays, nothing comes in)
        const size_t row = (size_t)(row0 + t_first + t);
        if (A.form == 0) {
          if (t < rows) {
            bb = ms_softplus(ms_gate_in<T>(A.g0, A.ldg0, A.gates_f32, row, head) + bias0);
            a = expf(-rate * bb);
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
            if (x == lane) { kept = kx; mine = m; }
          }
          if (t < rows) { a = expf(kept - mine); bb = expf(gi - mine); fl = expf(-mine); }
        }
        if (t < chunk) scalars[(ch & 1) * chunk + t] = make_float4(a, bb, fl, 0.f);
      }
    };
    form_chunk(0);
    for (int ch = 0; ch < n_chunks; ++ch) {
      __syncthreads();
      if (ch + 1 < n_chunks) form_chunk(ch + 1);
    }
    if (A.form == 1 && A.write_state)
      for (int j = j0 + lane; j < j_end; j += 32) ms[j] = m;
    return;
  }

  // ---- the columns ----------------------------------------------------------------------------------------
  const int grp = head / (H / A.G);
  const T* q = (const T*)A.q + (size_t)grp * dk;
  const T* k = (const T*)A.k + (size_t)grp * dk;
  const T* v = (const T*)A.v + (size_t)head * dv;
  // what no copy writes, in every stage: key channels beyond the head (zero), the normaliser's value (one) and what lies
  // behind it (zero)
  {
    const int extra_k = QW - dk, v_first = min(VTp, max(0, dv - j0)), extra_v = VTp - v_first, per = 2 * extra_k + extra_v;
    if (per > 0)
      for (int e = tid; e < MS_STAGES * chunk * per; e += n_compute) {
        const int t = e / per, s = t / chunk, r = t - s * chunk;
        int x = e - t * per;
        T* base = stages + (size_t)s * stage_elems;
        if (x < extra_k) base[(size_t)r * QW + dk + x] = from_f32<T>(0.f);
        else if ((x -= extra_k) < extra_k) base[(size_t)(chunk + r) * QW + dk + x] = from_f32<T>(0.f);
        else {
          x += v_first - extra_k;
          base[(size_t)2 * chunk * QW + (size_t)r * VTp + x] = from_f32<T>(j0 + x == dv ? 1.f : 0.f);
        }
      }
  }
  float2 s[J][DC / 2];
  ms_load_state<DC, J>(s, st, dk, l, jc, j_end, ctx > 0);
  const float skip = A.skip ? A.skip[head] : 0.f, q_scale = A.q_scale;
  pdl_wait();
  // a chunk's rows of q, k (the group's) and v (the tile's): pieces of 16 bytes, a thread keeps to one place of the row
  const int pk = dk / VEC, pv = min(VT, max(0, dv - j0)) / VEC, per = 2 * pk + pv;
  const int at_once = max(1, n_compute / max(1, per)), my_row = per <= n_compute ? tid / max(1, per) : 0;
  auto issue = [&](int ch) {
    if (ch < n_chunks) {
      T* base = stages + (size_t)(ch % MS_STAGES) * stage_elems;
      const int t_first = ch * chunk, rows = min(chunk, n - t_first);
      if (A.vec) {
        if (my_row < at_once)
          for (int x = per <= n_compute ? tid - my_row * per : tid; x < per; x += n_compute) {
            const T* src; T* dst; long ld; int pitch;
            if (x < pk) { src = q + x * VEC; ld = A.ldq; dst = base + x * VEC; pitch = QW; }
            else if (x < 2 * pk) { src = k + (x - pk) * VEC; ld = A.ldk; dst = base + (size_t)chunk * QW + (x - pk) * VEC; pitch = QW; }
            else { src = v + j0 + (x - 2 * pk) * VEC; ld = A.ldv; dst = base + (size_t)2 * chunk * QW + (x - 2 * pk) * VEC; pitch = VTp; }
            src += (size_t)(row0 + t_first + my_row) * ld;
            dst += my_row * pitch;
            const long src_step = (long)at_once * ld;
            const int dst_step = at_once * pitch;
            for (int t = my_row; t < chunk; t += at_once, dst += dst_step) {
              ms_cp_async16(dst, t < rows ? src : q, t < rows);
              src += src_step;
            }
          }
      } else {
        const int ev = min(VT, max(0, dv - j0)), pe = 2 * dk + ev;
        for (int e = tid; e < chunk * pe; e += n_compute) {
          const int t = e / pe;
          int x = e - t * pe;
          const size_t row = (size_t)(row0 + t_first + t);
          const bool in = t < rows;
          if (x < dk) base[(size_t)t * QW + x] = in ? q[row * A.ldq + x] : from_f32<T>(0.f);
          else if ((x -= dk) < dk) base[(size_t)(chunk + t) * QW + x] = in ? k[row * A.ldk + x] : from_f32<T>(0.f);
          else {
            x -= dk;
            base[(size_t)2 * chunk * QW + (size_t)t * VTp + x] = in ? v[row * A.ldv + j0 + x] : from_f32<T>(0.f);
          }
        }
      }
    }
    asm volatile("cp.async.commit_group;\n" ::: "memory");
  };
  for (int ch = 0; ch < MS_STAGES - 1; ++ch) issue(ch);
  const size_t o_ld = (size_t)H * dv;
  for (int ch = 0; ch < n_chunks; ++ch) {
    asm volatile("cp.async.wait_group %0;\n" :: "n"(MS_STAGES - 2) : "memory");
    __syncthreads();                                    // the chunk and its scalars are there; nobody reads the stage that is filled next
    issue(ch + MS_STAGES - 1);
    const int rows = min(chunk, n - ch * chunk);
    const T* base = stages + (size_t)(ch % MS_STAGES) * stage_elems;
    const T* qp = base + l * DC;
    const T* kp = base + (size_t)chunk * QW + l * DC;
    const T* vp = base + (size_t)2 * chunk * QW + cg * J;
    const float4* sc = scalars + (ch & 1) * chunk;
    const size_t row = (size_t)(row0 + ch * chunk);
    for (int t0 = 0; t0 < rows; t0 += TURN) {
      constexpr int NV = TURN * J;
      float val[NV];                                    // [token][column]
#pragma unroll
      for (int t = 0; t < TURN; ++t) {
        const float2 ab = *reinterpret_cast<const float2*>(sc + t0 + t);
        float2 qf[DC / 2], kf[DC / 2];
        float vv[J], u[J], acc[J];
        ms_pairs<DC>(qp + (size_t)(t0 + t) * QW, qf);
        ms_pairs<DC>(kp + (size_t)(t0 + t) * QW, kf);
        ms_values<J>(vp + (size_t)(t0 + t) * VTp, vv);
#pragma unroll
        for (int j = 0; j < J; ++j) u[j] = ab.y * vv[j];
        ms_token<DC, J>(s, qf, kf, u, ab.x, acc);
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
          const float y = val[i] * q_scale;
          if (col < dv) A.out[(row + t0 + t) * o_ld + (size_t)head * dv + col] = A.skip ? fmaf(skip, to_f32(vp[(size_t)(t0 + t) * VTp + j]), y) : y;
          else A.den[(row + t0 + t) * H + head] = fmaxf(fabsf(y), sc[t0 + t].z) + A.den_eps;
        }
      }
    }
  }
  if (A.write_state) ms_store_state<DC, J>(s, st, dk, l, jc, j_end);
}

// A step of single tokens: one token a request.
template <typename T, int DC, int J, int L>
__global__ void __launch_bounds__(ms_threads_max(J))
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
  float2 qf[DC / 2], kf[DC / 2];
#pragma unroll
  for (int i = 0; i < DC / 2; ++i) {
    const int c = l * DC + 2 * i;
    qf[i] = make_float2(c < dk ? to_f32(q[c]) : 0.f, c + 1 < dk ? to_f32(q[c + 1]) : 0.f);
    kf[i] = make_float2(c < dk ? to_f32(k[c]) : 0.f, c + 1 < dk ? to_f32(k[c + 1]) : 0.f);
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
      const float y = acc[j] * A.q_scale;
      if (col < dv) A.out[row * ((size_t)H * dv) + (size_t)head * dv + col] = A.skip ? fmaf(skip, vf[j], y) : y;
      else A.den[row * H + head] = fmaxf(fabsf(y), fl) + A.den_eps;
    }
  }
  if (A.write_state) {
    ms_store_state<DC, J>(s, st, dk, l, jc, j_end);
    // (every thread of the CTA has read its m; the CTA's columns are its own)
    if (A.form == 1) { __syncthreads(); for (int j = j0 + threadIdx.x; j < j_end; j += blockDim.x) ms[j] = m; }
  }
}

// The columns of a CTA: as many as its threads hold at most, fewer where the grid would leave SMs idle.
static int ms_threads(long units, int dvx, int L, int J) {
  int threads = ms_threads_max(J);
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
  const int VEC = 16 / (int)sizeof(T);
  const size_t token = (size_t)MS_STAGES * (2 * L * DC + (A.VT + VEC - 1) / VEC * VEC) * sizeof(T) + 2 * sizeof(float4);
  int chunk = 32;
  while (chunk > ms_turn(J) && (chunk * token > MS_SMEM_MAX || chunk / 2 >= max_q_len)) chunk >>= 1;
  const size_t smem = chunk * token;
  if (smem > MS_SMEM_MAX) QE_REFUSE("memory_scan: key size %d needs %zu bytes of shared memory", A.dk, smem);
  A.chunk = chunk;
  A.vec = A.dk % VEC == 0 && A.dv % VEC == 0 && A.VT % VEC == 0 && A.ldq % VEC == 0 && A.ldk % VEC == 0 && A.ldv % VEC == 0 &&
          (((uintptr_t)A.q | (uintptr_t)A.k | (uintptr_t)A.v) & 15) == 0;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(memory_scan_kernel<T, DC, J, L>, cudaFuncAttributeMaxDynamicSharedMemorySize, MS_SMEM_MAX);
    if (e != cudaSuccess) QE_REFUSE("memory_scan: shared memory: %s", cudaGetErrorString(e));
    configured = true;
  }
  qe_launch(memory_scan_kernel<T, DC, J, L>, grid, dim3(threads + 32), smem, stream, A);
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
  // Prompt portions in bfloat16 that fill the SMs only once: two columns a thread and twice the warps (latencies overlap);
  // otherwise four columns a thread (fewer conversions and loads for the same state).  The bits are the same.
  const bool few = max_q_len > 1 && dtype == QE_DTYPE_BF16 && DC == 8 && (long)R * H * ((A.dvx + 31) / 32) < 256;
#define MSL_L(TT, JJ) do { switch (L) { \
      case 1: return ms_launch<TT, 8, JJ, 1>(A, R, max_q_len, stream); case 2: return ms_launch<TT, 8, JJ, 2>(A, R, max_q_len, stream); \
      case 4: return ms_launch<TT, 8, JJ, 4>(A, R, max_q_len, stream); case 8: return ms_launch<TT, 8, JJ, 8>(A, R, max_q_len, stream); \
      case 16: return ms_launch<TT, 8, JJ, 16>(A, R, max_q_len, stream); default: return ms_launch<TT, 8, JJ, 32>(A, R, max_q_len, stream); } } while (0)
#define MSL(TT) do { \
    if (DC == 8) MSL_L(TT, 4); \
    switch (L) { case 16: return ms_launch<TT, 32, 1, 16>(A, R, max_q_len, stream); default: return ms_launch<TT, 32, 1, 32>(A, R, max_q_len, stream); } \
  } while (0)
  if (few) MSL_L(__nv_bfloat16, 2);
  if (dtype == QE_DTYPE_F32) MSL(float);
  if (dtype == QE_DTYPE_BF16) MSL(__nv_bfloat16);
#undef MSL
#undef MSL_L
  QE_REFUSE("memory_scan: unknown dtype %d", dtype);
}
