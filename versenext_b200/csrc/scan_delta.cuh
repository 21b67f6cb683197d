// Gated delta rule with one decay per key channel; the state S [dim, vdim] of a head is carried in fp32.
//
//   S <- g * S (row-wise) ; u = beta (v - S^T k) ; S <- S + k u^T ; o = S^T q
//
// The columns of S are independent of one another, so a column is the unit of parallelism; a group of lanes holds some
// columns in registers (rows spread over the lanes) and runs over the sequence's new tokens, while the next tokens'
// q, k, g, v are already being copied to shared memory.
// State layout [slot][R][head][vdim][dim] (a column is contiguous); ring of states as in scan_mamba.cuh.
#pragma once
#include "gemm_mma.cuh"
#include "rows.cuh"

struct DeltaRuleArgs {
  // scan inputs
  const float* q = nullptr;      // [M, KH * d] unit vectors, q times d^-1/2
  const float* k = nullptr;
  const float* v = nullptr;      // [M, H * vd]
  const float* g = nullptr;      // [M, H * d] decay factors
  const float* beta = nullptr;   // [M, H]
  float* o = nullptr;            // [M, H * vd]
  float* state = nullptr;
  int R = 2, H = 0, KH = 0, d = 0, vd = 0;
  Rows rows;
};

// what surrounds the recurrence
struct DeltaIn {
  Src src;                       // projection: q | k | v | beta | a1 | g1 columns
  int H = 0, KH = 0, d = 0, vd = 0, ra = 0, rg = 0, ra_ld = 0, rg_ld = 0;
  int col_b = 0, col_a = 0, col_g = 0;
  float* q = nullptr; float* k = nullptr; float* v = nullptr; float* beta = nullptr;
  void* low_a = nullptr; void* low_g = nullptr;    // [M, ra_ld], [M, rg_ld] storage dtype
  Rows rows;
  int pending = 1;
};

constexpr float UNIT_EPS = 1e-6f;   // inside the root of the unit norm of q and k

// Convolution + silu of q, k, v; unit vectors of q and k; beta; the two low-rank factors in the storage dtype.
// One warp per (RB rows, unit): units 0 .. KH-1 q heads, then KH k heads, H v heads, and one for the rest.
// grid (2 KH + H + 1, ceil(M / (8 RB))), block (32, 8)
template <typename T, int NC, int RB>      // NC: channels per lane (d, vd <= 32 NC)
__global__ void __launch_bounds__(256) delta_inputs_kernel(ConvIn<T> in, DeltaIn a) {
  const int lane = threadIdx.x, unit = blockIdx.x;
  int row = (blockIdx.y * 8 + threadIdx.y) * RB;
  const int last = min(row + RB, a.rows.M);
  const bool is_v = unit >= 2 * a.KH, is_k = !is_v && unit >= a.KH;
  const int w = is_v ? a.vd : a.d;
  const int c0 = is_v ? 2 * a.KH * a.d + (unit - 2 * a.KH) * a.vd : unit * a.d;
  while (row < last) {                                  // stretches of one entry
    if (unit == 2 * a.KH + a.H) {
      for (int h = lane; h < a.H; h += 32) a.beta[(long long)row * a.H + h] = sigmoid_f(a.src.get(row, a.col_b + h));
      for (int j = lane; j < a.ra_ld; j += 32)
        reinterpret_cast<T*>(a.low_a)[(long long)row * a.ra_ld + j] = from_f<T>(j < a.ra ? a.src.get(row, a.col_a + j) : 0.f);
      for (int j = lane; j < a.rg_ld; j += 32)
        reinterpret_cast<T*>(a.low_g)[(long long)row * a.rg_ld + j] = from_f<T>(j < a.rg ? a.src.get(row, a.col_g + j) : 0.f);
      ++row;
      continue;
    }
    int slot, r0, n, start;
    a.rows.entry(a.rows.entry_of(row), &slot, &r0, &n, &start);
    const int first = row, end = min(last, r0 + n);
    float val[RB][NC];
#pragma unroll (NC > 4 ? 1 : NC)             // wide heads: the convolution's code once
    for (int i = 0; i < NC; ++i) {
      const int j = lane + 32 * i;
      float v[RB];
#pragma unroll
      for (int r = 0; r < RB; ++r) v[r] = 0.f;
      if (j < w) {
        if constexpr (RB > 1) {                  // filters of at most four taps
          in.template run<RB>(first, end, r0, start, slot, c0 + j, v);
        } else {
          float cur;
          v[0] = in.at(first, r0, start, slot, c0 + j, &cur);
        }
      }
#pragma unroll
      for (int r = 0; r < RB; ++r) val[r][i] = v[r];
    }
    if (n <= a.pending)
      for (int r = first; r < end; ++r)
        for (int j = lane; j < w; j += 32) in.keep(slot, start + r - r0, c0 + j, in.src.get(r, in.col0 + c0 + j));
#pragma unroll
    for (int r = 0; r < RB; ++r) {
      if (first + r >= end) break;
      float* dst;
      float f = 1.f;
      if (is_v) {
        dst = a.v + (long long)(first + r) * a.H * a.vd + (unit - 2 * a.KH) * a.vd;
      } else {
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < NC; ++i) ss += val[r][i] * val[r][i];
        f = 1.f / sqrtf(warp_sum(ss) + UNIT_EPS);
        if (!is_k) f *= 1.f / sqrtf((float)a.d);
        dst = (is_k ? a.k : a.q) + (long long)(first + r) * a.KH * a.d + (is_k ? unit - a.KH : unit) * a.d;
      }
#pragma unroll
      for (int i = 0; i < NC; ++i)
        if (lane + 32 * i < w) dst[lane + 32 * i] = val[r][i] * f;
    }
    row = end;
  }
}

// g = exp(-exp(A_log_h) softplus(g + dt_bias)), in place over [M, H * d];  decay_rate[h] = exp(A_log_h)
static __global__ void __launch_bounds__(256) delta_decay_kernel(float* __restrict__ g, const float* __restrict__ decay_rate,
                                                          const float* __restrict__ dt_bias, long long total, int H, int d) {
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i >= total) return;
  const int c = (int)(i % ((long long)H * d));
  g[i] = expf(-decay_rate[c / d] * softplus_f(g[i] + dt_bias[c]));
}

// o / rms(o) over vdim * w * sigmoid(gate), one warp per (row, head).  grid ceil(M H / 8)
template <typename T>
__global__ void __launch_bounds__(256) delta_out_kernel(const float* __restrict__ o, const float* __restrict__ gate,
                                                        const float* __restrict__ w, T* __restrict__ out, long long n_heads,
                                                        int vd, float eps) {
  const long long i = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (i >= n_heads) return;
  const float* oi = o + i * vd;
  float ss = 0.f;
  for (int j = lane; j < vd; j += 32) ss += oi[j] * oi[j];
  const float r = sqrtf(warp_sum(ss) / (float)vd + eps);
  for (int j = lane; j < vd; j += 32) out[i * vd + j] = from_f<T>(oi[j] / r * w[j] * sigmoid_f(gate[i * vd + j]));
}

// One-token kernel: eight lanes share a column; rows of it held by a lane: register 4 i + e <-> row 32 i + 4 li + e (so that eight lanes read 128 contiguous
// bytes of q, k, g, and of a state column)

template <int DK>
__device__ __forceinline__ void delta_col_load(const float* col, int d, int li, bool ok, float (&S)[DK]) {
#pragma unroll
  for (int i = 0; i < DK / 4; ++i) {
    const int r = 32 * i + 4 * li;
    if (ok && r + 3 < d && (d & 3) == 0) {
      const float4 t = *reinterpret_cast<const float4*>(col + r);
      S[4 * i] = t.x; S[4 * i + 1] = t.y; S[4 * i + 2] = t.z; S[4 * i + 3] = t.w;
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e) S[4 * i + e] = (ok && r + e < d) ? col[r + e] : 0.f;
    }
  }
}
template <int DK>
__device__ __forceinline__ void delta_col_store(float* col, int d, int li, const float (&S)[DK]) {
#pragma unroll
  for (int i = 0; i < DK / 4; ++i) {
    const int r = 32 * i + 4 * li;
    if (r + 3 < d && (d & 3) == 0) {
      *reinterpret_cast<float4*>(col + r) = make_float4(S[4 * i], S[4 * i + 1], S[4 * i + 2], S[4 * i + 3]);
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (r + e < d) col[r + e] = S[4 * i + e];
    }
  }
}
// one token of NP columns (the lane's rows of each); o[p] receives the lane's part of the read-out
template <int DK, int NP>
__device__ __forceinline__ void delta_cols_step(float (&S)[NP][DK], const float* q, const float* k, const float* g, int li,
                                                const float (&v)[NP], float beta, float (&o)[NP]) {
  float dot[NP];
#pragma unroll
  for (int p = 0; p < NP; ++p) dot[p] = 0.f;
#pragma unroll
  for (int i = 0; i < DK / 4; ++i) {
    const float4 gv = *reinterpret_cast<const float4*>(g + 32 * i + 4 * li);
    const float4 kv = *reinterpret_cast<const float4*>(k + 32 * i + 4 * li);
#pragma unroll
    for (int p = 0; p < NP; ++p) {
      S[p][4 * i] *= gv.x; S[p][4 * i + 1] *= gv.y; S[p][4 * i + 2] *= gv.z; S[p][4 * i + 3] *= gv.w;
      dot[p] = fmaf(S[p][4 * i], kv.x, dot[p]); dot[p] = fmaf(S[p][4 * i + 1], kv.y, dot[p]);
      dot[p] = fmaf(S[p][4 * i + 2], kv.z, dot[p]); dot[p] = fmaf(S[p][4 * i + 3], kv.w, dot[p]);
    }
  }
#pragma unroll
  for (int p = 0; p < NP; ++p) {
    dot[p] += __shfl_xor_sync(0xffffffffu, dot[p], 1);
    dot[p] += __shfl_xor_sync(0xffffffffu, dot[p], 2);
    dot[p] += __shfl_xor_sync(0xffffffffu, dot[p], 4);
    dot[p] = beta * (v[p] - dot[p]);
    o[p] = 0.f;
  }
#pragma unroll
  for (int i = 0; i < DK / 4; ++i) {
    const float4 kv = *reinterpret_cast<const float4*>(k + 32 * i + 4 * li);
    const float4 qv = *reinterpret_cast<const float4*>(q + 32 * i + 4 * li);
#pragma unroll
    for (int p = 0; p < NP; ++p) {
      S[p][4 * i] = fmaf(kv.x, dot[p], S[p][4 * i]); S[p][4 * i + 1] = fmaf(kv.y, dot[p], S[p][4 * i + 1]);
      S[p][4 * i + 2] = fmaf(kv.z, dot[p], S[p][4 * i + 2]); S[p][4 * i + 3] = fmaf(kv.w, dot[p], S[p][4 * i + 3]);
      o[p] = fmaf(S[p][4 * i], qv.x, o[p]); o[p] = fmaf(S[p][4 * i + 1], qv.y, o[p]);
      o[p] = fmaf(S[p][4 * i + 2], qv.z, o[p]); o[p] = fmaf(S[p][4 * i + 3], qv.w, o[p]);
    }
  }
}

// 4 or 16 bytes from global to shared memory, asynchronously
template <int VEC>
__device__ __forceinline__ void cp_async_f(float* s, const float* g) {
  const unsigned a = (unsigned)__cvta_generic_to_shared(s);
  if (VEC == 4) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(a), "l"(g));
  else asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(a), "l"(g));
}

// ---- the scan over new tokens --------------------------------------------------------------------------------------
// Sixteen lanes share NC columns of the state, each with RPL rows of all of them, so that what a lane reads of q, k and g
// serves NC columns.  The NC partial sums of a dot product are reduced by halving: after log2(NC) exchanges every lane is
// left with one column's sum, the remaining exchanges complete it.  Rows are handled in pairs (two fp32 products or
// sums in one instruction).  Register 4 i + e <-> row 64 i + 4 li + e.
__device__ __forceinline__ unsigned long long f2_pack(float x, float y) {
  unsigned long long r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(x), "f"(y));
  return r;
}
__device__ __forceinline__ float f2_sum(unsigned long long v) {
  float x, y;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(v));
  return x + y;
}
__device__ __forceinline__ unsigned long long f2_mul(unsigned long long a, unsigned long long b) {
  unsigned long long r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ unsigned long long f2_fma(unsigned long long a, unsigned long long b, unsigned long long c) {
  unsigned long long r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
// sum of v[c] over the sixteen lanes of a group: the lane returns the total of column delta_scan_col<NC>(li)
template <int NC> __device__ __forceinline__ int delta_scan_col(int li) { return li / (16 / NC); }
template <int NC>
__device__ __forceinline__ float group_sum(float (&v)[NC], int li) {
#pragma unroll
  for (int half = NC / 2, bit = 8; half >= 1; half >>= 1, bit >>= 1) {
    const bool up = li & bit;
#pragma unroll
    for (int c = 0; c < half; ++c) {
      const float give = up ? v[c] : v[c + half], keep = up ? v[c + half] : v[c];
      v[c] = keep + __shfl_xor_sync(0xffffffffu, give, bit);
    }
  }
  float s = v[0];
#pragma unroll
  for (int bit = 8 / NC; bit >= 1; bit >>= 1) s += __shfl_xor_sync(0xffffffffu, s, bit);
  return s;
}

// RPL rows per lane (d <= 16 RPL); NC columns per group; VEC 4 when d and vd are multiples of 4; W warps.
// grid (ceil(vd / (2 NC W)), H, n_ent), 32 W threads
template <int RPL, int NC, int VEC, int W>
__global__ void __launch_bounds__(32 * W) delta_scan_kernel(DeltaRuleArgs a) {
  constexpr int DP = 16 * RPL, CT = RPL > 8 ? 4 : 8, COLS = 2 * NC * W, THREADS = 32 * W;
  typedef unsigned long long u64;
  __shared__ __align__(16) float s_q[2][CT][DP], s_k[2][CT][DP], s_g[2][CT][DP], s_v[2][CT][COLS];
  __shared__ float s_b[2][CT], s_o[CT][COLS];
  int slot, r0, n, start;
  a.rows.entry(blockIdx.z, &slot, &r0, &n, &start);
  if (n <= 0) return;
  const int tid = threadIdx.x, lane = tid & 31, h = blockIdx.y, kh = h / (a.H / a.KH), c0 = blockIdx.x * COLS;
  const int li = lane & 15, gcol = (tid >> 4) * NC;    // lane of the group; the group's first column in the CTA
  const int mine = gcol + delta_scan_col<NC>(li);      // the column whose sums this lane ends up with
  const int d = a.d, vd = a.vd, nv = min(COLS, vd - c0);
  for (int i = tid; i < 2 * CT * DP; i += THREADS) (&s_q[0][0][0])[i] = (&s_k[0][0][0])[i] = (&s_g[0][0][0])[i] = 0.f;
  for (int i = tid; i < 2 * CT * COLS; i += THREADS) (&s_v[0][0][0])[i] = 0.f;
  __syncthreads();
  u64 S[NC][RPL / 2];
  const long long one = (long long)vd * d;
  const bool vec = (d & 3) == 0;
  const float* st_in = a.state + (((long long)slot * a.R + start % a.R) * a.H + h) * one;
#pragma unroll
  for (int c = 0; c < NC; ++c)
#pragma unroll
    for (int i = 0; i < RPL / 4; ++i) {
      const int r = 64 * i + 4 * li;
      const float* p = st_in + (long long)(c0 + gcol + c) * d + r;
      const bool ok = start > 0 && c0 + gcol + c < vd;
      float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
      if (ok && vec && r < d) t = *reinterpret_cast<const float4*>(p);
      else if (ok) {
        if (r < d) t.x = p[0];
        if (r + 1 < d) t.y = p[1];
        if (r + 2 < d) t.z = p[2];
        if (r + 3 < d) t.w = p[3];
      }
      S[c][2 * i] = f2_pack(t.x, t.y);
      S[c][2 * i + 1] = f2_pack(t.z, t.w);
    }
  auto store_state = [&](int pos) {
    float* st = a.state + (((long long)slot * a.R + pos % a.R) * a.H + h) * one;
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
      for (int i = 0; i < RPL / 4; ++i) {
        const int r = 64 * i + 4 * li;
        if (c0 + gcol + c >= vd || r >= d) continue;
        float* p = st + (long long)(c0 + gcol + c) * d + r;
        float4 t;
        asm("mov.b64 {%0, %1}, %2;" : "=f"(t.x), "=f"(t.y) : "l"(S[c][2 * i]));
        asm("mov.b64 {%0, %1}, %2;" : "=f"(t.z), "=f"(t.w) : "l"(S[c][2 * i + 1]));
        if (vec) *reinterpret_cast<float4*>(p) = t;
        else {
          p[0] = t.x;
          if (r + 1 < d) p[1] = t.y;
          if (r + 2 < d) p[2] = t.z;
          if (r + 3 < d) p[3] = t.w;
        }
      }
  };
  auto fetch = [&](int t0, int buf) {
    const int m = min(CT, n - t0);
    const int per = d / VEC;
    for (int i = tid; i < m * per; i += THREADS) {
      const int t = i / per, j = (i % per) * VEC;
      const long long row = r0 + t0 + t;
      cp_async_f<VEC>(&s_q[buf][t][j], a.q + row * a.KH * d + kh * d + j);
      cp_async_f<VEC>(&s_k[buf][t][j], a.k + row * a.KH * d + kh * d + j);
      cp_async_f<VEC>(&s_g[buf][t][j], a.g + row * a.H * d + h * d + j);
    }
    const int pv = nv / VEC;
    for (int i = tid; i < m * pv; i += THREADS) {
      const int t = i / pv, j = (i % pv) * VEC;
      cp_async_f<VEC>(&s_v[buf][t][j], a.v + (long long)(r0 + t0 + t) * a.H * vd + h * vd + c0 + j);
    }
    if (tid < m) cp_async_f<1>(&s_b[buf][tid], a.beta + (long long)(r0 + t0 + tid) * a.H + h);
    mma_detail::cp_async_commit();
  };
  const bool snap = n <= a.R - 1;
  fetch(0, 0);
  for (int t0 = 0, buf = 0; t0 < n; t0 += CT, buf ^= 1) {
    if (t0 + CT < n) { fetch(t0 + CT, buf ^ 1); mma_detail::cp_async_wait<1>(); }
    else mma_detail::cp_async_wait<0>();
    __syncthreads();
    const int m = min(CT, n - t0);
    // The read-out sums of a token are finished together with the next token's first sums, and the next token's operands
    // are fetched under them: the recurrence itself (sum, exchange, update) is what is left on the critical path.
    u64 gg[RPL / 2], kk[RPL / 2], qq[RPL / 2];
    float part[NC], late[NC], vb, bb;
    auto operands = [&](int t) {
#pragma unroll
      for (int i = 0; i < RPL / 4; ++i) {
        const ulonglong2 g2 = *reinterpret_cast<const ulonglong2*>(&s_g[buf][t][64 * i + 4 * li]);
        const ulonglong2 k2 = *reinterpret_cast<const ulonglong2*>(&s_k[buf][t][64 * i + 4 * li]);
        const ulonglong2 q2 = *reinterpret_cast<const ulonglong2*>(&s_q[buf][t][64 * i + 4 * li]);
        gg[2 * i] = g2.x; gg[2 * i + 1] = g2.y; kk[2 * i] = k2.x; kk[2 * i + 1] = k2.y; qq[2 * i] = q2.x; qq[2 * i + 1] = q2.y;
      }
      vb = s_v[buf][t][mine];
      bb = s_b[buf][t];
    };
    operands(0);
    auto token = [&](int t, bool has_late) {
      {
        u64 acc[NC];
#pragma unroll
        for (int i = 0; i < RPL / 2; ++i)
#pragma unroll
          for (int c = 0; c < NC; ++c) {
            S[c][i] = f2_mul(S[c][i], gg[i]);
            acc[c] = i ? f2_fma(S[c][i], kk[i], acc[c]) : f2_mul(S[c][0], kk[0]);
          }
#pragma unroll
        for (int c = 0; c < NC; ++c) part[c] = f2_sum(acc[c]);
      }
      const float dot = group_sum<NC>(part, li);
      if (has_late) {
        const float o = group_sum<NC>(late, li);
        if ((li & (16 / NC - 1)) == 0) s_o[t - 1][mine] = o;
      }
      const float u = bb * (vb - dot);
      u64 uc[NC], k0[RPL / 2], q0[RPL / 2];
#pragma unroll
      for (int i = 0; i < RPL / 2; ++i) { k0[i] = kk[i]; q0[i] = qq[i]; }
      operands(min(t + 1, CT - 1));
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        const float x = __shfl_sync(0xffffffffu, u, (lane & 16) + c * (16 / NC));
        uc[c] = f2_pack(x, x);
      }
      u64 acc[NC];
#pragma unroll
      for (int i = 0; i < RPL / 2; ++i)
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          S[c][i] = f2_fma(k0[i], uc[c], S[c][i]);
          acc[c] = i ? f2_fma(S[c][i], q0[i], acc[c]) : f2_mul(S[c][0], q0[0]);
        }
#pragma unroll
      for (int c = 0; c < NC; ++c) late[c] = f2_sum(acc[c]);
    };
    if (!snap && m == CT) {
      token(0, false);
#pragma unroll
      for (int t = 1; t < CT; ++t) token(t, true);
    } else {
      for (int t = 0; t < m; ++t) {
        token(t, t > 0);
        if (snap) store_state(start + t0 + t + 1);
      }
    }
    {
      const float o = group_sum<NC>(late, li);
      if ((li & (16 / NC - 1)) == 0) s_o[m - 1][mine] = o;
    }
    __syncthreads();
    for (int i = tid; i < m * COLS; i += THREADS) {
      const int t = i / COLS, j = i % COLS;
      if (j < nv) a.o[(long long)(r0 + t0 + t) * a.H * vd + h * vd + c0 + j] = s_o[t][j];
    }
  }
  if (!snap) store_state(start + n);
}

// One new token per sequence, everything between the two projections in one kernel: convolutions, unit norms, beta,
// both low-rank products, decay, state update, read-out, norm and gate.  One CTA per (row, head).
template <typename T>
struct DeltaStepArgs {
  ConvIn<T> conv;
  DeltaIn in;                    // src, sizes and column offsets
  const T* w_a = nullptr;        // [H * d, ra_ld]
  const T* w_g = nullptr;        // [H * vd, rg_ld]
  const float* decay_rate = nullptr; const float* dt_bias = nullptr; const float* norm_w = nullptr;
  float* state = nullptr;
  int R = 2;
  float eps = 0.f;
  T* out = nullptr;              // [M, H * vd]
};

// dot of a weight row (ld entries, zero-padded, a multiple of 8) with a vector in shared memory, by `parts` lanes
template <typename T>
__device__ __forceinline__ float low_rank_dot(const T* w, const float* s, int ld, int part, int parts) {
  float acc = 0.f;
  if (sizeof(T) == 2) {
#pragma unroll 4
    for (int j = part * 8; j < ld; j += parts * 8) {
      const uint4 u = *reinterpret_cast<const uint4*>(w + j);
      const float4 x = *reinterpret_cast<const float4*>(s + j), y = *reinterpret_cast<const float4*>(s + j + 4);
      const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
      const float2 f0 = __bfloat1622float2(h[0]), f1 = __bfloat1622float2(h[1]), f2 = __bfloat1622float2(h[2]), f3 = __bfloat1622float2(h[3]);
      acc = fmaf(f0.x, x.x, acc); acc = fmaf(f0.y, x.y, acc); acc = fmaf(f1.x, x.z, acc); acc = fmaf(f1.y, x.w, acc);
      acc = fmaf(f2.x, y.x, acc); acc = fmaf(f2.y, y.y, acc); acc = fmaf(f3.x, y.z, acc); acc = fmaf(f3.y, y.w, acc);
    }
  } else {
    for (int j = part; j < ld; j += parts) acc = fmaf(to_f<T>(w[j]), s[j], acc);
  }
  return acc;
}

// NP: columns a lane takes at a time (the state of 64 NP columns is requested before anything else, so that it arrives
// under the convolutions and the low-rank products).  Shared memory: 3 DP + 3 vd + ra_ld + rg_ld floats.  grid (H, M)
constexpr int DELTA_STEP_THREADS = 512;
template <typename T, int DK, int NP>
__global__ void __launch_bounds__(DELTA_STEP_THREADS, 2) delta_step_kernel(DeltaStepArgs<T> a) {
  constexpr int DP = 8 * DK, TH = DELTA_STEP_THREADS, CP = TH / 8, RP = TH / 4;   // columns, low-rank rows per pass
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[TH / 32], s_misc[2];
  const DeltaIn& in = a.in;
  const int d = in.d, vd = in.vd, H = in.H, KH = in.KH;
  float *s_q = sm, *s_k = s_q + DP, *s_g = s_k + DP, *s_a = s_g + DP, *s_w = s_a + in.ra_ld, *s_v = s_w + in.rg_ld,
        *s_o = s_v + vd, *s_gate = s_o + vd;
  const int tid = threadIdx.x, h = blockIdx.x, row = blockIdx.y, kh = h / (H / KH);
  int slot, r0, n, start;
  in.rows.entry(in.rows.entry_of(row), &slot, &r0, &n, &start);
  const int cl = tid >> 3, li = tid & 7;
  const long long one = (long long)vd * d;
  const float* st_in = a.state + (((long long)slot * a.R + start % a.R) * H + h) * one;
  float* st_out = a.state + (((long long)slot * a.R + (start + 1) % a.R) * H + h) * one;
  float S[NP][DK];
#pragma unroll
  for (int p = 0; p < NP; ++p)
    delta_col_load<DK>(st_in + (long long)(cl + CP * p) * d, d, li, start > 0 && cl + CP * p < vd, S[p]);
  // inputs of this head
  const bool first = h % (H / KH) == 0;              // the group's first head keeps the shared q / k inputs
  // columns q | k | v (convolved) and a1 | g1 (as they are); one pass, small code: the kernel's instructions are fetched
  // anew at every step of a large model
  const int n_conv = 2 * d + vd, n_all = n_conv + in.ra + in.rg;
  const int taps = a.conv.taps, C = a.conv.C, RC = a.conv.RC;
  T* ring = a.conv.ring + (long long)slot * RC * C;
  for (int i = tid; i < n_all; i += TH) {
    int c;
    float* dst;
    if (i < d) { c = kh * d + i; dst = s_q + i; }
    else if (i < 2 * d) { c = (KH + kh) * d + i - d; dst = s_k + i - d; }
    else if (i < n_conv) { c = 2 * KH * d + h * vd + i - 2 * d; dst = s_v + i - 2 * d; }
    else if (i < n_conv + in.ra) { c = in.col_a + i - n_conv; dst = s_a + i - n_conv; }
    else { c = in.col_g + i - n_conv - in.ra; dst = s_w + i - n_conv - in.ra; }
    float past = 0.f, w0 = 1.f;
    if (i < n_conv) {                                // what came before is requested ahead of the projection's slices
      const float* wc = a.conv.w + (long long)c * taps;
      w0 = wc[taps - 1];
#pragma unroll 3
      for (int j = 1; j < taps; ++j)
        past = fmaf(start >= j ? to_f<T>(ring[(long long)((start - j) % RC) * C + c]) : 0.f, wc[taps - 1 - j], past);
    }
    float x = round_to<T>(in.src.get(row, c));
    if (i < n_conv) {
      if (first || i >= 2 * d) ring[(long long)(start % RC) * C + c] = from_f<T>(x);
      x = silu_as<T>(fmaf(x, w0, past));
    }
    *dst = x;
  }
  for (int j = d + tid; j < DP; j += TH) s_q[j] = s_k[j] = 0.f;
  for (int j = in.ra + tid; j < in.ra_ld; j += TH) s_a[j] = 0.f;
  for (int j = in.rg + tid; j < in.rg_ld; j += TH) s_w[j] = 0.f;
  if (tid == 0) s_misc[0] = sigmoid_f(in.src.get(row, in.col_b + h));
  __syncthreads();
  // unit norms: warp 0 takes q, warp 1 takes k
  const int warp = tid >> 5, lane = tid & 31;
  if (warp < 2) {
    float* s = warp ? s_k : s_q;
    float ss = 0.f;
    for (int j = lane; j < d; j += 32) ss += s[j] * s[j];
    float f = 1.f / sqrtf(warp_sum(ss) + UNIT_EPS);
    if (!warp) f *= 1.f / sqrtf((float)d);
    for (int j = lane; j < d; j += 32) s[j] *= f;
  }
  // decays of the key channels, then gates of the value columns: four lanes per row of the low-rank matrices
  const int nd = (DP + RP - 1) / RP * RP;
#pragma unroll 1
  for (int j0 = 0; j0 < nd + vd; j0 += RP) {
    const int jj = j0 + (tid >> 2);
    const bool dec = j0 < nd;
    const int j = dec ? jj : jj - nd;
    const T* w = dec ? a.w_a + (long long)(h * d + j) * in.ra_ld : a.w_g + (long long)(h * vd + j) * in.rg_ld;
    float acc = j < (dec ? d : vd) ? low_rank_dot<T>(w, dec ? s_a : s_w, dec ? in.ra_ld : in.rg_ld, tid & 3, 4) : 0.f;
    acc += __shfl_xor_sync(0xffffffffu, acc, 1);
    acc += __shfl_xor_sync(0xffffffffu, acc, 2);
    if ((tid & 3) == 0) {
      if (dec && j < DP) s_g[j] = j < d ? expf(-a.decay_rate[h] * softplus_f(acc + a.dt_bias[h * d + j])) : 0.f;
      if (!dec && j < vd) s_gate[j] = sigmoid_f(acc);
    }
  }
  __syncthreads();
  const float beta = s_misc[0];
  float ss = 0.f;
  for (int c0 = 0; c0 < vd; c0 += CP * NP) {
    float v[NP], o[NP];
#pragma unroll
    for (int p = 0; p < NP; ++p) {
      const int c = c0 + cl + CP * p;
      if (c0 > 0) delta_col_load<DK>(st_in + (long long)c * d, d, li, start > 0 && c < vd, S[p]);
      v[p] = c < vd ? s_v[c] : 0.f;
    }
    delta_cols_step<DK, NP>(S, s_q, s_k, s_g, li, v, beta, o);
#pragma unroll
    for (int p = 0; p < NP; ++p) {
      const int c = c0 + cl + CP * p;
      o[p] += __shfl_xor_sync(0xffffffffu, o[p], 1);
      o[p] += __shfl_xor_sync(0xffffffffu, o[p], 2);
      o[p] += __shfl_xor_sync(0xffffffffu, o[p], 4);
      if (c < vd) {
        if (li == 0) { s_o[c] = o[p]; ss += o[p] * o[p]; }
        delta_col_store<DK>(st_out + (long long)c * d, d, li, S[p]);
      }
    }
  }
  ss = warp_sum(ss);
  if (lane == 0) red[warp] = ss;
  __syncthreads();                                   // also publishes s_o
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < TH / 32; ++i) ss += red[i];
  const float r = sqrtf(ss / (float)vd + a.eps);
  for (int j = tid; j < vd; j += TH)
    a.out[(long long)row * H * vd + h * vd + j] = from_f<T>(s_o[j] / r * a.norm_w[j] * s_gate[j]);
}

template <typename T> int32_t vn_delta_inputs(vn_ctx* ctx, const ConvIn<T>& conv, const DeltaIn& in);
template <typename T> int32_t vn_delta_step(vn_ctx* ctx, const DeltaStepArgs<T>& a);
int32_t vn_delta_scan(vn_ctx* ctx, const DeltaRuleArgs& a);
