// Gated delta rule with one decay per key channel; the state S [dim, vdim] of a head is carried in fp32.
//
//   S <- g * S (row-wise) ; u = beta (v - S^T k) ; S <- S + k u^T ; o = S^T q
//
// The columns of S are independent of one another, so a column is the unit of parallelism: eight lanes share one (each
// holds DK of its rows in registers), a CTA of 128 threads takes 16 columns of one head of one sequence and runs over
// the sequence's new tokens, with the next CT tokens' q, k, g, v already being copied to shared memory.
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
// One warp per (row, unit): units 0 .. KH-1 q heads, then KH k heads, H v heads, and one for the rest.
// grid (2 KH + H + 1, ceil(M / 8)), block (32, 8)
template <typename T, int NC>      // NC: channels per lane (d, vd <= 32 NC)
__global__ void __launch_bounds__(256) delta_inputs_kernel(ConvIn<T> in, DeltaIn a) {
  const int row = blockIdx.y * 8 + threadIdx.y, lane = threadIdx.x, unit = blockIdx.x;
  if (row >= a.rows.M) return;
  int slot, r0, n, start;
  a.rows.entry(a.rows.entry_of(row), &slot, &r0, &n, &start);
  if (unit == 2 * a.KH + a.H) {
    for (int h = lane; h < a.H; h += 32) a.beta[(long long)row * a.H + h] = sigmoid_f(a.src.get(row, a.col_b + h));
    for (int j = lane; j < a.ra_ld; j += 32)
      reinterpret_cast<T*>(a.low_a)[(long long)row * a.ra_ld + j] = from_f<T>(j < a.ra ? a.src.get(row, a.col_a + j) : 0.f);
    for (int j = lane; j < a.rg_ld; j += 32)
      reinterpret_cast<T*>(a.low_g)[(long long)row * a.rg_ld + j] = from_f<T>(j < a.rg ? a.src.get(row, a.col_g + j) : 0.f);
    return;
  }
  const bool is_v = unit >= 2 * a.KH;
  const int w = is_v ? a.vd : a.d;
  const int c0 = is_v ? 2 * a.KH * a.d + (unit - 2 * a.KH) * a.vd : unit * a.d;
  float val[NC], ss = 0.f;
#pragma unroll
  for (int i = 0; i < NC; ++i) {
    const int j = lane + 32 * i;
    val[i] = 0.f;
    if (j < w) {
      float cur;
      val[i] = in.at(row, r0, start, slot, c0 + j, &cur);
      if (n <= a.pending) in.keep(slot, start + row - r0, c0 + j, cur);
      ss += val[i] * val[i];
    }
  }
  float* dst;
  float f = 1.f;
  if (is_v) {
    dst = a.v + (long long)row * a.H * a.vd + (unit - 2 * a.KH) * a.vd;
  } else {
    const bool is_k = unit >= a.KH;
    f = 1.f / sqrtf(warp_sum(ss) + UNIT_EPS);
    if (!is_k) f *= 1.f / sqrtf((float)a.d);
    dst = (is_k ? a.k : a.q) + (long long)row * a.KH * a.d + (is_k ? unit - a.KH : unit) * a.d;
  }
#pragma unroll
  for (int i = 0; i < NC; ++i)
    if (lane + 32 * i < w) dst[lane + 32 * i] = val[i] * f;
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

// rows of a column held by a lane: register 4 i + e <-> row 32 i + 4 li + e (so that eight lanes read 128 contiguous
// bytes of q, k, g, and of a state column)
constexpr int DR_COLS = 16;

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
// one token of one column (the lane's rows): returns the lane's part of o
template <int DK>
__device__ __forceinline__ float delta_col_step(float (&S)[DK], const float* q, const float* k, const float* g, int li,
                                                float v, float beta) {
  float d0 = 0.f, d1 = 0.f;
#pragma unroll
  for (int i = 0; i < DK / 4; ++i) {
    const float4 gv = *reinterpret_cast<const float4*>(g + 32 * i + 4 * li);
    const float4 kv = *reinterpret_cast<const float4*>(k + 32 * i + 4 * li);
    S[4 * i] *= gv.x; S[4 * i + 1] *= gv.y; S[4 * i + 2] *= gv.z; S[4 * i + 3] *= gv.w;
    d0 = fmaf(S[4 * i], kv.x, d0); d1 = fmaf(S[4 * i + 1], kv.y, d1);
    d0 = fmaf(S[4 * i + 2], kv.z, d0); d1 = fmaf(S[4 * i + 3], kv.w, d1);
  }
  float dot = d0 + d1;
  dot += __shfl_xor_sync(0xffffffffu, dot, 1);
  dot += __shfl_xor_sync(0xffffffffu, dot, 2);
  dot += __shfl_xor_sync(0xffffffffu, dot, 4);
  const float u = beta * (v - dot);
  float o0 = 0.f, o1 = 0.f;
#pragma unroll
  for (int i = 0; i < DK / 4; ++i) {
    const float4 kv = *reinterpret_cast<const float4*>(k + 32 * i + 4 * li);
    const float4 qv = *reinterpret_cast<const float4*>(q + 32 * i + 4 * li);
    S[4 * i] = fmaf(kv.x, u, S[4 * i]); S[4 * i + 1] = fmaf(kv.y, u, S[4 * i + 1]);
    S[4 * i + 2] = fmaf(kv.z, u, S[4 * i + 2]); S[4 * i + 3] = fmaf(kv.w, u, S[4 * i + 3]);
    o0 = fmaf(S[4 * i], qv.x, o0); o1 = fmaf(S[4 * i + 1], qv.y, o1);
    o0 = fmaf(S[4 * i + 2], qv.z, o0); o1 = fmaf(S[4 * i + 3], qv.w, o1);
  }
  return o0 + o1;
}

// 4 or 16 bytes from global to shared memory, asynchronously
template <int VEC>
__device__ __forceinline__ void cp_async_f(float* s, const float* g) {
  const unsigned a = (unsigned)__cvta_generic_to_shared(s);
  if (VEC == 4) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(a), "l"(g));
  else asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(a), "l"(g));
}

// DK rows per lane (d <= 8 DK); VEC 4 when d and vd are multiples of 4.  grid (ceil(vd / 16), H, n_ent), 128 threads
template <int DK, int VEC>
__global__ void __launch_bounds__(128) delta_scan_kernel(DeltaRuleArgs a) {
  constexpr int DP = 8 * DK, CT = DK > 16 ? 4 : 8;
  __shared__ __align__(16) float s_q[2][CT][DP], s_k[2][CT][DP], s_g[2][CT][DP], s_v[2][CT][DR_COLS];
  __shared__ float s_b[2][CT], s_o[CT][DR_COLS];
  int slot, r0, n, start;
  a.rows.entry(blockIdx.z, &slot, &r0, &n, &start);
  if (n <= 0) return;
  const int tid = threadIdx.x, h = blockIdx.y, kh = h / (a.H / a.KH), c0 = blockIdx.x * DR_COLS;
  const int cl = tid >> 3, li = tid & 7;              // column of the CTA, lane of the column
  const bool ok = c0 + cl < a.vd;
  const int d = a.d, vd = a.vd, nv = min(DR_COLS, vd - c0);
  for (int i = tid; i < 2 * CT * DP; i += 128) (&s_q[0][0][0])[i] = (&s_k[0][0][0])[i] = (&s_g[0][0][0])[i] = 0.f;
  for (int i = tid; i < 2 * CT * DR_COLS; i += 128) (&s_v[0][0][0])[i] = 0.f;
  __syncthreads();
  float S[DK];
  const long long one = (long long)vd * d;
  delta_col_load<DK>(a.state + (((long long)slot * a.R + start % a.R) * a.H + h) * one + (long long)(c0 + cl) * d, d, li,
                     ok && start > 0, S);
  auto store_state = [&](int p) {
    if (ok) delta_col_store<DK>(a.state + (((long long)slot * a.R + p % a.R) * a.H + h) * one + (long long)(c0 + cl) * d, d, li, S);
  };
  auto fetch = [&](int t0, int buf) {
    const int m = min(CT, n - t0);
    const int per = d / VEC;
    for (int i = tid; i < m * per; i += 128) {
      const int t = i / per, j = (i % per) * VEC;
      const long long row = r0 + t0 + t;
      cp_async_f<VEC>(&s_q[buf][t][j], a.q + row * a.KH * d + kh * d + j);
      cp_async_f<VEC>(&s_k[buf][t][j], a.k + row * a.KH * d + kh * d + j);
      cp_async_f<VEC>(&s_g[buf][t][j], a.g + row * a.H * d + h * d + j);
    }
    const int pv = nv / VEC;
    for (int i = tid; i < m * pv; i += 128) {
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
#pragma unroll 2
    for (int t = 0; t < m; ++t) {
      float o = delta_col_step<DK>(S, s_q[buf][t], s_k[buf][t], s_g[buf][t], li, s_v[buf][t][cl], s_b[buf][t]);
      o += __shfl_xor_sync(0xffffffffu, o, 1);
      o += __shfl_xor_sync(0xffffffffu, o, 2);
      o += __shfl_xor_sync(0xffffffffu, o, 4);
      if (li == 0) s_o[t][cl] = o;
      if (snap) store_state(start + t0 + t + 1);
    }
    __syncthreads();
    for (int i = tid; i < m * DR_COLS; i += 128) {
      const int t = i / DR_COLS, j = i % DR_COLS;
      if (j < nv) a.o[(long long)(r0 + t0 + t) * a.H * vd + h * vd + c0 + j] = s_o[t][j];
    }
  }
  if (!snap) store_state(start + n);
}

// One new token per sequence, everything between the two projections in one kernel: convolutions, unit norms, beta,
// both low-rank products, decay, state update, read-out, norm and gate.  One CTA (256 threads) per (row, head).
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
    for (int j = part * 8; j < ld; j += parts * 8) {
      const uint4 u = *reinterpret_cast<const uint4*>(w + j);
      const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const float2 f = __bfloat1622float2(h[q]);
        acc = fmaf(f.x, s[j + 2 * q], acc);
        acc = fmaf(f.y, s[j + 2 * q + 1], acc);
      }
    }
  } else {
    for (int j = part; j < ld; j += parts) acc = fmaf(to_f<T>(w[j]), s[j], acc);
  }
  return acc;
}

// shared memory: 3 DP + 2 vd + ra_ld + rg_ld floats.  grid (H, M)
template <typename T, int DK>
__global__ void __launch_bounds__(256) delta_step_kernel(DeltaStepArgs<T> a) {
  constexpr int DP = 8 * DK;
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[8], s_misc[2];
  const DeltaIn& in = a.in;
  const int d = in.d, vd = in.vd, H = in.H, KH = in.KH;
  float *s_q = sm, *s_k = s_q + DP, *s_g = s_k + DP, *s_a = s_g + DP, *s_w = s_a + in.ra_ld, *s_v = s_w + in.rg_ld, *s_o = s_v + vd;
  const int tid = threadIdx.x, h = blockIdx.x, row = blockIdx.y, kh = h / (H / KH);
  int slot, r0, n, start;
  in.rows.entry(in.rows.entry_of(row), &slot, &r0, &n, &start);
  // this thread's first column of the state: requested before anything else
  const int cl = tid >> 3, li = tid & 7;
  const long long one = (long long)vd * d;
  const float* st_in = a.state + (((long long)slot * a.R + start % a.R) * H + h) * one;
  float* st_out = a.state + (((long long)slot * a.R + (start + 1) % a.R) * H + h) * one;
  float S[DK];
  delta_col_load<DK>(st_in + (long long)cl * d, d, li, start > 0 && cl < vd, S);
  // inputs of this head
  const bool first = h % (H / KH) == 0;              // the group's first head keeps the shared q / k inputs
  for (int i = tid; i < 2 * DP + vd; i += 256) {
    float cur, v = 0.f;
    if (i < 2 * DP) {
      const int j = i % DP;
      if (j < d) {
        const int c = (i < DP ? 0 : KH * d) + kh * d + j;
        v = a.conv.at(row, r0, start, slot, c, &cur);
        if (first) a.conv.keep(slot, start, c, cur);
      }
      (i < DP ? s_q : s_k)[j] = v;
    } else {
      const int c = 2 * KH * d + h * vd + (i - 2 * DP);
      s_v[i - 2 * DP] = a.conv.at(row, r0, start, slot, c, &cur);
      a.conv.keep(slot, start, c, cur);
    }
  }
  for (int j = tid; j < in.ra_ld; j += 256) s_a[j] = j < in.ra ? round_to<T>(in.src.get(row, in.col_a + j)) : 0.f;
  for (int j = tid; j < in.rg_ld; j += 256) s_w[j] = j < in.rg ? round_to<T>(in.src.get(row, in.col_g + j)) : 0.f;
  if (tid == 0) s_misc[0] = sigmoid_f(in.src.get(row, in.col_b + h));
  __syncthreads();
  // unit norms: warp 0 takes q, warp 1 takes k; the others already start on the decays
  const int warp = tid >> 5, lane = tid & 31;
  if (warp < 2) {
    float* s = warp ? s_k : s_q;
    float ss = 0.f;
    for (int j = lane; j < d; j += 32) ss += s[j] * s[j];
    float f = 1.f / sqrtf(warp_sum(ss) + UNIT_EPS);
    if (!warp) f *= 1.f / sqrtf((float)d);
    for (int j = lane; j < d; j += 32) s[j] *= f;
  }
  for (int j0 = 0; j0 < DP; j0 += 64) {               // four lanes per key channel
    const int j = j0 + (tid >> 2);
    float acc = j < d ? low_rank_dot<T>(a.w_a + (long long)(h * d + j) * in.ra_ld, s_a, in.ra_ld, tid & 3, 4) : 0.f;
    acc += __shfl_xor_sync(0xffffffffu, acc, 1);
    acc += __shfl_xor_sync(0xffffffffu, acc, 2);
    if ((tid & 3) == 0 && j < DP)
      s_g[j] = j < d ? expf(-a.decay_rate[h] * softplus_f(acc + a.dt_bias[h * d + j])) : 0.f;
  }
  __syncthreads();
  const float beta = s_misc[0];
  for (int c0 = 0; c0 < vd; c0 += 32) {
    const int c = c0 + cl;
    const bool ok = c < vd;
    if (c0 > 0) delta_col_load<DK>(st_in + (long long)c * d, d, li, start > 0 && ok, S);
    float o = delta_col_step<DK>(S, s_q, s_k, s_g, li, ok ? s_v[c] : 0.f, beta);
    o += __shfl_xor_sync(0xffffffffu, o, 1);
    o += __shfl_xor_sync(0xffffffffu, o, 2);
    o += __shfl_xor_sync(0xffffffffu, o, 4);
    if (ok) {
      if (li == 0) s_o[c] = o;
      delta_col_store<DK>(st_out + (long long)c * d, d, li, S);
    }
  }
  __syncthreads();
  float ss = 0.f;
  for (int j = tid; j < vd; j += 256) ss += s_o[j] * s_o[j];
  const float r = sqrtf(block_sum256(ss, red) / (float)vd + a.eps);
  for (int j0 = 0; j0 < vd; j0 += 64) {
    const int j = j0 + (tid >> 2);
    float acc = j < vd ? low_rank_dot<T>(a.w_g + (long long)(h * vd + j) * in.rg_ld, s_w, in.rg_ld, tid & 3, 4) : 0.f;
    acc += __shfl_xor_sync(0xffffffffu, acc, 1);
    acc += __shfl_xor_sync(0xffffffffu, acc, 2);
    if ((tid & 3) == 0 && j < vd)
      a.out[(long long)row * H * vd + h * vd + j] = from_f<T>(s_o[j] / r * a.norm_w[j] * sigmoid_f(acc));
  }
}

template <typename T> int32_t vn_delta_inputs(vn_ctx* ctx, const ConvIn<T>& conv, const DeltaIn& in);
template <typename T> int32_t vn_delta_step(vn_ctx* ctx, const DeltaStepArgs<T>& a);
int32_t vn_delta_scan(vn_ctx* ctx, const DeltaRuleArgs& a);
