// Selective scan (Mamba) with a state per (channel, state index) carried in fp32 per sequence.
//
//   S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n ;  y_c = sum_n S[c, n] C_n + D_c x_c ;  out = y * silu(z)
//
// A recurrence runs over the tokens of one sequence; its parallelism is channels x sequences.  A few lanes share a
// channel (each holds some of its states in registers), a CTA takes 32 channels of one sequence and stages the per-token inputs of CT tokens in shared memory while the next CT tokens are on their way.
//
// State ring: the state after p tokens of slot s lives at ring index p mod R.  A forward of n rows leaves the state
// after every row when n is small enough to be cut back (n <= R - 1), otherwise the last one only; committing k rows
// then is a change of the sequence's length and nothing else.
#pragma once
#include "rows.cuh"
#include <type_traits>

struct MambaArgs {
  const float* dt = nullptr;     // [M, inner] W_dt dt, before the bias (scan); unused by the step kernel
  const void* xc = nullptr;      // [M, inner] convolved input, storage dtype
  const void* z = nullptr;       // [M, inner] storage dtype
  Src p;                         // W_x x: [dt: dt_cols | B: state | C: state]
  int dt_cols = 0, dt_rank = 0;  // padded width of the dt part, and its true width
  const void* w_dt = nullptr;    // [inner, dt_cols] storage dtype (step kernel)
  const float* dt_bias = nullptr;
  const float* A = nullptr;      // [inner, state] -exp(A_log)
  const float* D = nullptr;
  float* state = nullptr;        // [slots][R][inner][state]
  int R = 2, inner = 0, nstate = 0;
  void* out = nullptr;           // [M, inner] storage dtype
  Rows rows;
};

// convolution of the x half, copy of the z half.  grid (ceil(inner / 32), ceil(M / (8 RB))), block (32, 8): a thread
// takes one channel of RB rows (8 for prompts, 1 when every entry has one row)
template <typename T, int RB>
__global__ void __launch_bounds__(256) mamba_conv_kernel(ConvIn<T> in, Rows rows, T* __restrict__ xc, T* __restrict__ z,
                                                         int pending) {
  const int c = blockIdx.x * 32 + threadIdx.x;
  int row = (blockIdx.y * 8 + threadIdx.y) * RB;
  const int last = min(row + RB, rows.M);
  if (c >= in.C) return;
  while (row < last) {                                 // stretches of one entry
    int slot, r0, n, start;
    rows.entry(rows.entry_of(row), &slot, &r0, &n, &start);
    const int first = row, end = min(last, r0 + n);
    float v[RB], zv[RB];
    in.src.template column<RB>(first, end, in.col0 + in.C + c, zv);
    if (RB > 1 && in.taps <= 4) {
      in.template run<RB>(first, end, r0, start, slot, c, v);
    } else {
#pragma unroll
      for (int r = 0; r < RB; ++r) {
        float cur;
        v[r] = first + r < end ? in.at(first + r, r0, start, slot, c, &cur) : 0.f;
      }
    }
    if (n <= pending)
      for (int r = first; r < end; ++r) in.keep(slot, start + r - r0, c, in.src.get(r, in.col0 + c));
#pragma unroll
    for (int r = 0; r < RB; ++r) {
      if (first + r >= end) break;
      xc[(long long)(first + r) * in.C + c] = from_f<T>(v[r]);
      z[(long long)(first + r) * in.C + c] = from_f<T>(zv[r]);
    }
    row = end;
  }
}

// the dt columns of W_x x as the operand of W_dt (padding columns zero).  grid M
template <typename T>
__global__ void cast_cols_kernel(Src src, int col0, int n, T* __restrict__ out, int ld) {
  for (int j = threadIdx.x; j < ld; j += blockDim.x)
    out[(long long)blockIdx.x * ld + j] = from_f<T>(j < n ? src.get(blockIdx.x, col0 + j) : 0.f);
}

constexpr int MAMBA_CH = 32, MAMBA_CT = 16;
constexpr float LOG2E = 1.4426950408889634f;       // exp(dt A) = 2^(dt (A log2 e))

// L lanes share a channel, NS states each (nstate <= L NS); 32 L threads.  grid (ceil(inner / 32), n_ent)
template <typename T, int NS, int L>
__global__ void __launch_bounds__(32 * L) mamba_scan_kernel(MambaArgs a) {
  constexpr int N4 = L * NS, THREADS = 32 * L, CT = MAMBA_CT, CH = MAMBA_CH;
  __shared__ float s_dt[2][CT][CH], s_x[2][CT][CH], s_y[CT][CH];
  __shared__ __align__(16) float s_b[2][CT][N4], s_c[2][CT][N4];
  int slot, r0, n, start;
  a.rows.entry(blockIdx.y, &slot, &r0, &n, &start);
  if (n <= 0) return;
  const int tid = threadIdx.x, ch = tid / L, l = tid % L;
  const int c0 = blockIdx.x * CH, c = c0 + ch;
  const bool c_ok = c < a.inner;
  const T* xc = reinterpret_cast<const T*>(a.xc);
  const T* zz = reinterpret_cast<const T*>(a.z);
  T* out = reinterpret_cast<T*>(a.out);

  float S[NS], A[NS];
  const float* st_in = a.state + ((long long)slot * a.R + start % a.R) * a.inner * a.nstate;
#pragma unroll
  for (int j = 0; j < NS; ++j) {
    const int i = l * NS + j;
    const bool ok = c_ok && i < a.nstate;
    A[j] = ok ? a.A[(long long)c * a.nstate + i] * LOG2E : 0.f;
    S[j] = (ok && start > 0) ? st_in[(long long)c * a.nstate + i] : 0.f;
  }
  auto store_state = [&](int p) {
    float* so = a.state + ((long long)slot * a.R + p % a.R) * a.inner * a.nstate;
#pragma unroll
    for (int j = 0; j < NS; ++j) {
      const int i = l * NS + j;
      if (c_ok && i < a.nstate) so[(long long)c * a.nstate + i] = S[j];
    }
  };

  // staging: thread -> (token ti + L k, channel tc) for the per-channel inputs, flat indices for B and C
  const int tc = tid & 31, ti = tid >> 5;
  const bool tc_ok = c0 + tc < a.inner;
  const float bias = tc_ok ? a.dt_bias[c0 + tc] : 0.f, Dc = tc_ok ? a.D[c0 + tc] : 0.f;
  constexpr int BI = (CT * N4 + THREADS - 1) / THREADS;
  float r_dt[CT / L], r_x[CT / L], r_z[CT / L], z_cur[CT / L], r_b[BI], r_c[BI];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int k = 0; k < CT / L; ++k) {
      const int t = t0 + ti + L * k;
      r_dt[k] = r_x[k] = r_z[k] = 0.f;
      if (t < n && tc_ok) {
        const long long o = (long long)(r0 + t) * a.inner + c0 + tc;
        r_dt[k] = a.dt[o]; r_x[k] = to_f<T>(xc[o]); r_z[k] = to_f<T>(zz[o]);
      }
    }
#pragma unroll
    for (int k = 0; k < BI; ++k) {
      const int f = tid + k * THREADS, t = t0 + f / N4, i = f % N4;
      r_b[k] = r_c[k] = 0.f;
      if (f < CT * N4 && t < n && i < a.nstate) {
        r_b[k] = a.p.get(r0 + t, a.dt_cols + i);
        r_c[k] = a.p.get(r0 + t, a.dt_cols + a.nstate + i);
      }
    }
  };
  auto stash = [&](int buf) {
#pragma unroll
    for (int k = 0; k < CT / L; ++k) {
      s_dt[buf][ti + L * k][tc] = softplus_f(r_dt[k] + bias);
      s_x[buf][ti + L * k][tc] = r_x[k];
      z_cur[k] = r_z[k];
    }
#pragma unroll
    for (int k = 0; k < BI; ++k) {
      const int f = tid + k * THREADS;
      if (f < CT * N4) { s_b[buf][f / N4][f % N4] = r_b[k]; s_c[buf][f / N4][f % N4] = r_c[k]; }
    }
  };
  const bool snap = n <= a.R - 1;
  fetch(0);
  for (int t0 = 0, buf = 0; t0 < n; t0 += CT, buf ^= 1) {
    stash(buf);
    __syncthreads();
    if (t0 + CT < n) fetch(t0 + CT);
    const int m = min(CT, n - t0);
    // G tokens at a time: everything that does not depend on the state first
    auto tokens = [&](int t, auto tag) {
      constexpr int G = decltype(tag)::value;
      __align__(16) float e[G][NS], bx[G][NS], cv[G][NS];
      float y[G];
#pragma unroll
      for (int q = 0; q < G; ++q) {
        const float d = s_dt[buf][t + q][ch], dx = d * s_x[buf][t + q][ch];
        if (NS % 4 == 0) {
#pragma unroll
          for (int j = 0; j < NS; j += 4) {
            *reinterpret_cast<float4*>(&bx[q][j]) = *reinterpret_cast<const float4*>(&s_b[buf][t + q][l * NS + j]);
            *reinterpret_cast<float4*>(&cv[q][j]) = *reinterpret_cast<const float4*>(&s_c[buf][t + q][l * NS + j]);
          }
        } else {
#pragma unroll
          for (int j = 0; j < NS; ++j) { bx[q][j] = s_b[buf][t + q][l * NS + j]; cv[q][j] = s_c[buf][t + q][l * NS + j]; }
        }
#pragma unroll
        for (int j = 0; j < NS; ++j) { e[q][j] = exp2f(d * A[j]); bx[q][j] *= dx; }
      }
#pragma unroll
      for (int q = 0; q < G; ++q) {
        y[q] = 0.f;
#pragma unroll
        for (int j = 0; j < NS; ++j) {
          S[j] = fmaf(e[q][j], S[j], bx[q][j]);
          y[q] = fmaf(S[j], cv[q][j], y[q]);
        }
      }
#pragma unroll
      for (int o = 1; o < L; o <<= 1)
#pragma unroll
        for (int q = 0; q < G; ++q) y[q] += __shfl_xor_sync(0xffffffffu, y[q], o);
      if (l == 0)
#pragma unroll
        for (int q = 0; q < G; ++q) s_y[t + q][ch] = y[q];
    };
    if (!snap && m == CT) {
      constexpr int G = NS <= 4 ? 4 : NS <= 8 ? 2 : 1;
#pragma unroll 1
      for (int t = 0; t < CT; t += G) tokens(t, std::integral_constant<int, G>());
    } else {
      for (int t = 0; t < m; ++t) {
        tokens(t, std::integral_constant<int, 1>());
        if (snap) store_state(start + t0 + t + 1);
      }
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < CT / L; ++k) {
      const int t = ti + L * k;
      if (t < m && tc_ok) {
        const float z = z_cur[k];
        const float y = s_y[t][tc] + Dc * s_x[buf][t][tc];
        out[(long long)(r0 + t0 + t) * a.inner + c0 + tc] = from_f<T>(y * silu_as<T>(z));
      }
    }
  }
  if (!snap) store_state(start + n);
}

// One new token per sequence: the dt projection, the state update and the gate in one kernel.  256 threads, 256 / L
// channels of one row; grid (ceil(inner / (256 / L)), M), shared memory (dt_cols + 2 nstate) floats
template <typename T, int NS, int L>
__global__ void __launch_bounds__(256) mamba_step_kernel(MambaArgs a) {
  extern __shared__ __align__(16) float s_p[];
  const int row = blockIdx.y;
  int slot, r0, n, start;
  a.rows.entry(a.rows.entry_of(row), &slot, &r0, &n, &start);
  const int tid = threadIdx.x, ch = tid / L, l = tid % L;
  const int c = blockIdx.x * (256 / L) + ch;
  const bool c_ok = c < a.inner;
  const int cc = c_ok ? c : a.inner - 1;               // lanes beyond the last channel go along without storing
  const long long o = (long long)row * a.inner + cc;
  const float x = to_f<T>(reinterpret_cast<const T*>(a.xc)[o]), z = to_f<T>(reinterpret_cast<const T*>(a.z)[o]);
  // the state and A do not depend on the projection: on their way while it is summed
  float S[NS], A[NS];
  const float* st_in = a.state + ((long long)slot * a.R + start % a.R) * a.inner * a.nstate;
#pragma unroll
  for (int j = 0; j < NS; ++j) {
    const int i = l * NS + j;
    const bool ok = c_ok && i < a.nstate;
    A[j] = ok ? a.A[(long long)c * a.nstate + i] * LOG2E : 0.f;
    S[j] = (ok && start > 0) ? st_in[(long long)c * a.nstate + i] : 0.f;
  }
  const int np = a.dt_cols + 2 * a.nstate;
  for (int j = tid; j < np; j += 256) {
    const float v = (j >= a.dt_rank && j < a.dt_cols) ? 0.f : a.p.get(row, j);
    s_p[j] = j < a.dt_cols ? round_to<T>(v) : v;      // the operand of W_dt is in the storage dtype, as in the scan route
  }
  __syncthreads();
  float acc = 0.f;
  if (c_ok) {
    const T* w = reinterpret_cast<const T*>(a.w_dt) + (long long)c * a.dt_cols;
    if (sizeof(T) == 2) {                             // dt_cols is a multiple of 8: 16-byte loads
#pragma unroll 4
      for (int j = l * 8; j < a.dt_cols; j += 8 * L) {
        const uint4 u = *reinterpret_cast<const uint4*>(w + j);
        const float4 x = *reinterpret_cast<const float4*>(s_p + j), y = *reinterpret_cast<const float4*>(s_p + j + 4);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
        const float2 f0 = __bfloat1622float2(h[0]), f1 = __bfloat1622float2(h[1]), f2 = __bfloat1622float2(h[2]), f3 = __bfloat1622float2(h[3]);
        acc = fmaf(f0.x, x.x, acc); acc = fmaf(f0.y, x.y, acc); acc = fmaf(f1.x, x.z, acc); acc = fmaf(f1.y, x.w, acc);
        acc = fmaf(f2.x, y.x, acc); acc = fmaf(f2.y, y.y, acc); acc = fmaf(f3.x, y.z, acc); acc = fmaf(f3.y, y.w, acc);
      }
    } else {
      for (int j = l; j < a.dt_cols; j += L) acc = fmaf(to_f<T>(w[j]), s_p[j], acc);
    }
  }
#pragma unroll
  for (int o = 1; o < L; o <<= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
  const float d = softplus_f(acc + a.dt_bias[cc]);
  float* so = a.state + ((long long)slot * a.R + (start + 1) % a.R) * a.inner * a.nstate;
  float y = 0.f;
#pragma unroll
  for (int j = 0; j < NS; ++j) {
    const int i = l * NS + j;
    if (i < a.nstate) {
      S[j] = fmaf(exp2f(d * A[j]), S[j], d * x * s_p[a.dt_cols + i]);
      y = fmaf(S[j], s_p[a.dt_cols + a.nstate + i], y);
      if (c_ok) so[(long long)c * a.nstate + i] = S[j];
    }
  }
#pragma unroll
  for (int q = 1; q < L; q <<= 1) y += __shfl_xor_sync(0xffffffffu, y, q);
  if (l == 0 && c_ok) reinterpret_cast<T*>(a.out)[o] = from_f<T>((y + a.D[c] * x) * silu_as<T>(z));
}

int32_t vn_mamba_scan(vn_ctx* ctx, const MambaArgs& a, bool bf16);
int32_t vn_mamba_step(vn_ctx* ctx, const MambaArgs& a, bool bf16);
