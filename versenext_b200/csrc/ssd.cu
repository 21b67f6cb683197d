// Kernels of ssd.cuh.
#include <algorithm>
#include <type_traits>

#include "ldmatrix.cuh"
#include "scan_delta.cuh"      // columns of a state in registers
#include "ssd.cuh"

namespace {

using bf16 = __nv_bfloat16;
constexpr float LOG2E = 1.4426950408889634f;
constexpr int SCAN_TH = 256, SCAN_COLS = SCAN_TH / 8;

// ---- inputs --------------------------------------------------------------------------------------------------------------
// grid (ceil(C / 32) + ceil(H / 32) [+ ceil(H P / 32): z], ceil(M / (8 RB))), block (32, 8): a thread takes one channel, one
// head's step size or one gate of RB rows
template <typename T, typename S, int RB>
__global__ void __launch_bounds__(256) ssd_inputs_kernel(ConvIn<T, S> in, SsdArgs a) {
  const int blocks = (in.C + 31) / 32;
  int row = (blockIdx.y * 8 + threadIdx.y) * RB;
  const int last = min(row + RB, a.rows.M);
  if ((int)blockIdx.x >= blocks) {
    const int h = ((int)blockIdx.x - blocks) * 32 + threadIdx.x, hp = (a.H + 31) / 32 * 32;
    if (h >= hp) {
      const int c = h - hp, n = a.inner();
      for (; c < n && row < last; ++row) reinterpret_cast<T*>(a.z)[(long long)row * n + c] = from_f<T>(in.src.get(row, c));
      return;
    }
    if (h >= a.H) return;
    const float bias = a.dt_bias[h];
    for (; row < last; ++row) a.dt[(long long)row * a.H + h] = softplus_f(in.src.get_rare(row, a.col_dt() + h) + bias);
    return;
  }
  const int c = blockIdx.x * 32 + threadIdx.x;
  if (c >= in.C) return;
  T* out = reinterpret_cast<T*>(a.xbc);
  while (row < last) {                                 // stretches of one entry
    int slot, r0, n, start;
    a.rows.entry(a.rows.entry_of(row), &slot, &r0, &n, &start);
    const int first = row, end = min(last, r0 + n);
    float v[RB];
    if (RB > 1 && in.taps <= 4) {
      in.template run<RB>(first, end, r0, start, slot, c, v);
    } else {
#pragma unroll
      for (int r = 0; r < RB; ++r) {
        float cur = 0.f;
        v[r] = first + r < end ? in.at(first + r, r0, start, slot, c, &cur) : 0.f;
        if (RB == 1 && n <= a.pending && in.taps > 1) in.keep(slot, start + first - r0, c, cur);
      }
    }
    if (RB > 1 && n <= a.pending && in.taps > 1)
      for (int r = first; r < end; ++r) in.keep(slot, start + r - r0, c, in.src.get_rare(r, in.col0 + c));
#pragma unroll
    for (int r = 0; r < RB; ++r) {
      if (first + r >= end) break;
      out[(long long)(first + r) * a.ld + c] = from_f<T>(v[r]);
    }
    row = end;
  }
}

// The same for many rows: four channels of RB rows per thread, `rep` times.  Filters of at most four taps; the number of
// channels, the first column and the pitches multiples of 4.  grid (ceil((C / 4 + H) / 256), ceil(M / (rep RB)))
template <typename T, int RB>
__global__ void __launch_bounds__(256) ssd_inputs4_kernel(ConvIn<T, Mat<T>> in, SsdArgs a, int rep) {
  const int it = blockIdx.x * 256 + threadIdx.x, quads = in.C / 4;
  int row = blockIdx.y * rep * RB;
  const int last = min(row + rep * RB, a.rows.M);
  if (it >= quads) {
    const int h = it - quads;
    if (h >= a.H) return;
    const float bias = a.dt_bias[h];
#pragma unroll 4
    for (; row < last; ++row) a.dt[(long long)row * a.H + h] = softplus_f(in.src.get(row, a.col_dt() + h) + bias);
    return;
  }
  const int c = it * 4;
  T* out = reinterpret_cast<T*>(a.xbc) + c;
  float w[4][4];
  in.filters4(c, w);
#pragma unroll 1
  while (row < last) {
    int slot, r0, n, start;
    a.rows.entry(a.rows.entry_of(row), &slot, &r0, &n, &start);
    const int end = min(min(last, row + RB), r0 + n);
    float4 v[RB];
    in.template run4<RB>(row, end, r0, start, slot, c, w, v);
#pragma unroll
    for (int r = 0; r < RB; ++r) {
      if (row + r >= end) break;
      store4(out + (long long)(row + r) * a.ld, v[r]);
      if (n <= a.pending && in.taps > 1)
        for (int e = 0; e < 4; ++e) in.keep(slot, start + row + r - r0, c + e, in.src.get(row + r, in.col0 + c + e));
    }
    row = end;
  }
}

// ---- token after token -------------------------------------------------------------------------------------------------------
// Eight lanes share a column of S; DK rows of it per lane (N <= 8 DK), NP columns per group.  A CTA runs over all rows of an
// entry with its columns in registers.  STEP: one row per entry, whose inputs are convolved here; the group's first head
// keeps the inputs of B and C.  grid (H * ceil(P / (32 NP)), n_ent)
template <typename T, typename S, int DK, int NP, bool STEP>
__global__ void __launch_bounds__(SCAN_TH) ssd_scan_kernel(ConvIn<T, S> in, SsdArgs a) {
  constexpr int DP = 8 * DK, COLS = SCAN_COLS * NP, NB = STEP ? 1 : 2;
  __shared__ __align__(16) float s_b[NB][DP], s_c[NB][DP];
  __shared__ float s_x[NB][COLS], s_dt[NB];
  const int tid = threadIdx.x, nb = (a.P + COLS - 1) / COLS, h = blockIdx.x / nb, cb = (blockIdx.x % nb) * COLS;
  const int N = a.N, P = a.P, cl = tid >> 3, li = tid & 7, inner = a.inner(), g = h / (a.H / a.G), nv = min(COLS, P - cb);
  int slot, r0, n, start;
  a.rows.entry(blockIdx.y, &slot, &r0, &n, &start);
  if (n <= 0) return;
  const long long one = (long long)P * N;
  const float* st_in = a.state + (((long long)slot * a.R + start % a.R) * a.H + h) * one;
  float St[NP][DK];
#pragma unroll
  for (int p = 0; p < NP; ++p) {
    const int c = cb + cl + SCAN_COLS * p;
    delta_col_load<DK>(st_in + (long long)c * N, N, li, start > 0 && c < P, St[p]);
  }
  const float A = a.A[h] * LOG2E, D = a.D[h];
  const bool snap = n <= a.R - 1;
  for (int j = N + tid; j < DP; j += SCAN_TH)
#pragma unroll
    for (int b = 0; b < NB; ++b) s_b[b][j] = s_c[b][j] = 0.f;
  const T* xbc = reinterpret_cast<const T*>(a.xbc);
#pragma unroll 1
  for (int t = 0; t < (STEP ? 1 : n); ++t) {
    const int buf = STEP ? 0 : t & 1;
    const long long row = r0 + t;
#pragma unroll 1
    for (int i = tid; i < 2 * N + nv + 1; i += SCAN_TH) {
      if (i == 2 * N + nv) {
        s_dt[buf] = STEP ? softplus_f(in.src.get_rare(row, a.col_dt() + h) + a.dt_bias[h]) : a.dt[row * a.H + h];
        break;
      }
      const int c = i < N ? inner + g * N + i : i < 2 * N ? inner + (a.G + g) * N + i - N : h * P + cb + i - 2 * N;
      float x;
      if constexpr (STEP) {
        float cur;
        x = round_to<T>(in.at((int)row, r0, start, slot, c, &cur));
        if (in.taps > 1 && (i >= 2 * N || (cb == 0 && h % (a.H / a.G) == 0))) in.keep(slot, start, c, cur);
      } else {
        x = to_f<T>(xbc[row * a.ld + c]);
      }
      float* dst = i < N ? &s_b[buf][i] : i < 2 * N ? &s_c[buf][i - N] : &s_x[buf][i - 2 * N];
      *dst = x;
    }
    __syncthreads();
    const float dt = s_dt[buf], dec = exp2f(A * dt);
    float o[NP], v[NP];
#pragma unroll
    for (int p = 0; p < NP; ++p) { o[p] = 0.f; v[p] = cl + SCAN_COLS * p < nv ? dt * s_x[buf][cl + SCAN_COLS * p] : 0.f; }
#pragma unroll
    for (int i = 0; i < DK / 4; ++i) {
      const float4 b4 = load4(&s_b[buf][32 * i + 4 * li]), c4 = load4(&s_c[buf][32 * i + 4 * li]);
      const float bb[4] = {b4.x, b4.y, b4.z, b4.w}, cc[4] = {c4.x, c4.y, c4.z, c4.w};
#pragma unroll
      for (int p = 0; p < NP; ++p)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          float& s = St[p][4 * i + e];
          s = fmaf(dec, s, bb[e] * v[p]);
          o[p] = fmaf(s, cc[e], o[p]);
        }
    }
    // lane p of a group finishes column p
    float mine = 0.f;
#pragma unroll
    for (int p = 0; p < NP; ++p) {
      o[p] += __shfl_xor_sync(0xffffffffu, o[p], 1);
      o[p] += __shfl_xor_sync(0xffffffffu, o[p], 2);
      o[p] += __shfl_xor_sync(0xffffffffu, o[p], 4);
      if (li == p) mine = o[p];
    }
    const int cm = cl + SCAN_COLS * li;
    if (li < NP && cm < nv) {
      const int col = h * P + cb + cm;
      reinterpret_cast<T*>(a.u)[row * inner + col] = from_f<T>((mine + D * s_x[buf][cm]) * silu_as<T>(in.src.get(row, col)));
    }
    if (snap || t == n - 1) {
      float* st = a.state + (((long long)slot * a.R + (start + t + 1) % a.R) * a.H + h) * one;
#pragma unroll
      for (int p = 0; p < NP; ++p) {
        const int c = cb + cl + SCAN_COLS * p;
        if (c < P) delta_col_store<DK>(st + (long long)c * N, N, li, St[p]);
      }
    }
  }
}

// One row per entry, inputs convolved: bound by the state's bytes, so no barrier and nothing in shared memory.  A CTA takes
// `heads` heads in turn, the next one's state on its way while this one's is updated; B and C stay in registers within a group.
// N, H P and the pitch multiples of 4.  grid (ceil(H / heads) * ceil(P / (32 NP)), n_ent)
template <typename T, int DK, int NP>
__global__ void __launch_bounds__(SCAN_TH, 2) ssd_token_kernel(SsdArgs a, Mat<T> z, int heads) {
  constexpr int COLS = SCAN_COLS * NP;
  const int tid = threadIdx.x, nb = (a.P + COLS - 1) / COLS, h0 = (blockIdx.x / nb) * heads, h1 = min(a.H, h0 + heads);
  const int N = a.N, P = a.P, li = tid & 7, c0 = (blockIdx.x % nb) * COLS + (tid >> 3), inner = a.inner(), per = a.H / a.G;
  int slot, row, n, start;
  a.rows.entry(blockIdx.y, &slot, &row, &n, &start);
  if (n <= 0) return;
  const long long one = (long long)P * N;
  const float* st_in = a.state + ((long long)slot * a.R + start % a.R) * a.H * one + (long long)c0 * N + 4 * li;
  float* st_out = a.state + ((long long)slot * a.R + (start + 1) % a.R) * a.H * one + (long long)c0 * N + 4 * li;
  const T* in = reinterpret_cast<const T*>(a.xbc) + (long long)row * a.ld;
  struct Head { float4 st[NP][DK / 4]; float x[NP], z, dt; };
  auto fetch = [&](int h, Head& f) {
#pragma unroll
    for (int p = 0; p < NP; ++p) {
      const int c = c0 + SCAN_COLS * p;
#pragma unroll
      for (int i = 0; i < DK / 4; ++i)
        f.st[p][i] = start > 0 && c < P && 32 * i + 4 * li < N ? load4(st_in + h * one + (long long)SCAN_COLS * p * N + 32 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
      f.x[p] = c < P ? to_f<T>(in[h * P + c]) : 0.f;
    }
    f.dt = a.dt[(long long)row * a.H + h];
    const int c = c0 + SCAN_COLS * li;
    f.z = li < NP && c < P ? z.get(row, h * P + c) : 0.f;
  };
  Head cur, next;
  fetch(h0, cur);
  float4 B[DK / 4], C[DK / 4];
  int group = -1;
#pragma unroll 1
  for (int h = h0; h < h1; ++h) {
    if (h + 1 < h1) fetch(h + 1, next);
    if (h / per != group) {
      group = h / per;
      const T* b = in + inner + group * N + 4 * li;
#pragma unroll
      for (int i = 0; i < DK / 4; ++i) {
        const bool ok = 32 * i + 4 * li < N;
        B[i] = ok ? load4(b + 32 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
        C[i] = ok ? load4(b + a.G * N + 32 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
    }
    const float dec = exp2f(a.A[h] * LOG2E * cur.dt), D = a.D[h];
    float mine = 0.f, xm = 0.f;
#pragma unroll
    for (int p = 0; p < NP; ++p) {
      const float v = cur.dt * cur.x[p];
      float o = 0.f;
#pragma unroll
      for (int i = 0; i < DK / 4; ++i) {
        float4& s = cur.st[p][i];
        s = make_float4(fmaf(dec, s.x, B[i].x * v), fmaf(dec, s.y, B[i].y * v), fmaf(dec, s.z, B[i].z * v), fmaf(dec, s.w, B[i].w * v));
        o = fmaf(s.x, C[i].x, fmaf(s.y, C[i].y, fmaf(s.z, C[i].z, fmaf(s.w, C[i].w, o))));
        if (c0 + SCAN_COLS * p < P && 32 * i + 4 * li < N) store4(st_out + h * one + (long long)SCAN_COLS * p * N + 32 * i, s);
      }
      o += __shfl_xor_sync(0xffffffffu, o, 1);
      o += __shfl_xor_sync(0xffffffffu, o, 2);
      o += __shfl_xor_sync(0xffffffffu, o, 4);
      if (li == p) { mine = o; xm = cur.x[p]; }
    }
    const int c = c0 + SCAN_COLS * li;
    if (li < NP && c < P) reinterpret_cast<T*>(a.u)[(long long)row * inner + h * P + c] = from_f<T>((mine + D * xm) * silu_as<T>(cur.z));
    cur = next;
  }
}

// columns per group: more fetch B and C fewer times, fewer make more CTAs
int scan_np(const vn_ctx* ctx, int H, int P, int N, int n_ent) {
  if (N > 128) return 1;
  for (int np : {4, 2})
    if (P > SCAN_COLS * np / 2 && (long long)n_ent * H * ceil_div(P, SCAN_COLS * np) >= 2 * ctx->sm_count) return np;
  return 1;
}

template <typename T, typename S, bool STEP>
int32_t launch_scan(vn_ctx* ctx, const ConvIn<T, S>& in, const SsdArgs& a) {
  const char* name = STEP ? "ssd_step_kernel" : "ssd_scan_kernel";
  const int np = scan_np(ctx, a.H, a.P, a.N, a.rows.n_ent);
  const dim3 grid(a.H * ceil_div(a.P, SCAN_COLS * np), a.rows.n_ent);
#define SCAN2(DK, NP) VN_LAUNCH_NAMED(ctx, name, (ssd_scan_kernel<T, S, DK, NP, STEP>), grid, SCAN_TH, 0, in, a)
#define SCAN(DK) do { if (np == 4) SCAN2(DK, 4); else if (np == 2) SCAN2(DK, 2); else SCAN2(DK, 1); } while (0)
  if (a.N <= 32) SCAN(4); else if (a.N <= 64) SCAN(8); else if (a.N <= 128) SCAN(16);
  else if (a.N <= 256) SCAN2(32, 1); else SCAN2(64, 1);
#undef SCAN
#undef SCAN2
  return VN_OK;
}

// ---- chunked kernel ------------------------------------------------------------------------------------------------------
// With L_i the sum of A dt up to token i of a chunk of CH tokens,
//   y_i = exp(L_i) S^T C_i + sum_{j <= i} exp(L_i - L_j) dt_j (C_i . B_j) x_j + D x_i ,
//   S <- exp(L_last) S + sum_j exp(L_last - L_j) dt_j B_j x_j^T .
// x, B and C are 16-bit values; what is fp32 by nature (the state, the decayed scores, the weighted x) enters a tensor-core
// product as three bf16 pieces that add up to it, so nothing of the recurrence is computed at less than fp32.
//
// CTA = four warps, 64 columns (of P) of one head; warp w keeps the state of columns 16 w .. 16 w + 15 transposed in its
// accumulators [16][N], which is also the layout its pieces have as the B operand of C S.
constexpr int CH = 64, CW = 4, VB = 16 * CW;

template <int DT> constexpr int chunk_smem(bool local) {
  const int q = 2 * CH * (DT + 8) * 2, v = 2 * CH * (VB + 8) * 2, p = CH * (CH + 4) * 4;
  return local ? q + v : 2 * q + v + p;
}

// two neighbouring gate values as they come from the projection
__device__ __forceinline__ float2 gate2(const Mat<bf16>& m, long long row, int col) {
  return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(m.p + row * m.ld + col));
}
__device__ __forceinline__ float2 gate2(const Src& m, long long row, int col) { return make_float2(m.get_rare(row, col), m.get_rare(row, col + 1)); }

// LOCAL: only the state a segment would end with if it began with nothing, to seg_state, and its decay (all but the last
// segment).  VEC: 16-byte copies.  grid (H * ceil(P / VB), segments, n_ent)
template <int DT, bool LOCAL, bool VEC, typename S>
__global__ void __launch_bounds__(32 * CW) ssd_chunk_kernel(SsdArgs a, S proj) {
  using namespace mma_detail;
  constexpr int LQ = DT + 8, LV = VB + 8, LP = CH + 4, TH = 32 * CW, NT = DT / 8;
  extern __shared__ __align__(16) unsigned char raw[];
  bf16* sK = reinterpret_cast<bf16*>(raw);                       // [2][CH][LQ] B
  bf16* sV = sK + 2 * CH * LQ;                                   // [2][CH][LV] x
  bf16* sQ = sV + 2 * CH * LV;                                   // [2][CH][LQ] C
  float* sP = reinterpret_cast<float*>(sQ + (LOCAL ? 0 : 2 * CH * LQ));   // [CH][LP]
  __shared__ __align__(16) float s_L[CH], s_dt[CH], s_w[CH];                   // exponents up to a token; step sizes; weights in the new state
  int slot, r0, n, start;
  a.rows.entry(blockIdx.z, &slot, &r0, &n, &start);
  const int seg = blockIdx.y, t_lo = seg * a.seg_len, t_hi = min(n, t_lo + a.seg_len);
  if (t_lo >= n) return;
  if (LOCAL && t_hi == n) return;                                // nobody starts behind the last piece
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int nvb = (a.P + VB - 1) / VB, h = blockIdx.x / nvb, cb = (blockIdx.x % nvb) * VB, N = a.N, P = a.P, inner = a.inner();
  const int nv = min(VB, P - cb), g = h / (a.H / a.G), kb = inner + g * N, kc = inner + (a.G + g) * N, kx = h * P + cb;
  const float A = a.A[h] * LOG2E, D = a.D[h];
  const bf16 zero = __float2bfloat16_rn(0.f);
  // zero what no fetch writes: states beyond N and columns beyond P
  for (int i = tid; i < 2 * CH * (DT - N); i += TH) {
    const int r = i / (DT - N), c = N + i % (DT - N);
    sK[r * LQ + c] = zero;
    if (!LOCAL) sQ[r * LQ + c] = zero;
  }
  for (int i = tid; i < 2 * CH * (VB - nv); i += TH) sV[(i / (VB - nv)) * LV + nv + i % (VB - nv)] = zero;
  const bf16* xbc = reinterpret_cast<const bf16*>(a.xbc);
  float dt_next[2];                                              // of tokens 2 lane and 2 lane + 1 (warp 0)
  auto fetch = [&](int t0, int buf) {
    const int m = min(CH, t_hi - t0);
    const bf16* base = xbc + (long long)(r0 + t0) * a.ld;
    if (VEC) {
      const int pd = N / 8, pv = nv / 8;
      for (int i = tid; i < CH * pd; i += TH) {
        const int r = i / pd, c = (i % pd) * 8;
        const bf16* src = base + (long long)(r < m ? r : 0) * a.ld + c;
        if (!LOCAL) cp_async16(sQ + (buf * CH + r) * LQ + c, src + kc, r < m);
        cp_async16(sK + (buf * CH + r) * LQ + c, src + kb, r < m);
      }
      for (int i = tid; i < CH * pv; i += TH) {
        const int r = i / pv, c = (i % pv) * 8;
        cp_async16(sV + (buf * CH + r) * LV + c, base + (long long)(r < m ? r : 0) * a.ld + kx + c, r < m);
      }
    } else {
      for (int i = tid; i < CH * N; i += TH) {
        const int r = i / N, c = i % N;
        const bf16* src = base + (long long)r * a.ld + c;
        if (!LOCAL) sQ[(buf * CH + r) * LQ + c] = r < m ? src[kc] : zero;
        sK[(buf * CH + r) * LQ + c] = r < m ? src[kb] : zero;
      }
      for (int i = tid; i < CH * nv; i += TH) {
        const int r = i / nv, c = i % nv;
        sV[(buf * CH + r) * LV + c] = r < m ? base[(long long)r * a.ld + kx + c] : zero;
      }
    }
    cp_async_commit();
    if (warp == 0)
#pragma unroll
      for (int e = 0; e < 2; ++e) dt_next[e] = 2 * lane + e < m ? a.dt[(long long)(r0 + t0 + 2 * lane + e) * a.H + h] : 0.f;
  };
  fetch(t_lo, 0);
  // St[j][0..1]: column cb + 16 warp + lane / 4, rows 8 j + 2 (lane % 4) + {0, 1}; [2..3]: column + 8
  const int g4 = lane >> 2, l2 = (lane & 3) * 2;
  const long long one = (long long)P * N;
  float St[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) St[j][e] = 0.f;
  auto add_state = [&](const float* st, float keep) {            // St = keep St + st
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int c = cb + 16 * warp + g4 + 8 * e;
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const int r = 8 * j + l2 + x;
          St[j][2 * e + x] = fmaf(keep, St[j][2 * e + x], c < P && r < N ? st[(long long)c * N + r] : 0.f);
        }
    }
  };
  auto store_state = [&](float* st) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int c = cb + 16 * warp + g4 + 8 * e;
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const int r = 8 * j + l2 + x;
          if (c < P && r < N) st[(long long)c * N + r] = St[j][2 * e + x];
        }
    }
  };
  auto piece = [&](int s) { return a.seg_state + (((long long)blockIdx.z * a.segments + s) * a.H + h) * one; };
  auto piece_decay = [&](int s) -> float& { return a.seg_decay[((long long)blockIdx.z * a.segments + s) * a.H + h]; };
  const float* initial = start > 0 ? a.state + (((long long)slot * a.R + start % a.R) * a.H + h) * one : nullptr;
  if (LOCAL) {
    if (seg == 0 && initial) {
      add_state(initial, 0.f);
      store_state(piece(a.segments - 1));
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) St[j][e] = 0.f;
    }
  } else {
    if (initial) add_state(n > a.seg_len ? piece(a.segments - 1) : initial, 0.f);
#pragma unroll 1
    for (int s = 0; s < seg; ++s) add_state(piece(s), exp2f(piece_decay(s)));
  }
  float total = 0.f;                                             // exponent of the segment's decay (LOCAL)
#pragma unroll 1
  for (int t0 = t_lo, buf = 0; t0 < t_hi; t0 += CH, buf ^= 1) {
    const int m = min(CH, t_hi - t0);
    if (warp == 0) {                                             // step sizes and running exponents; flat beyond the last token
      const float e0 = A * dt_next[0], e1 = A * dt_next[1];
      float sum = e0 + e1;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float up = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += up;
      }
      const float last = __shfl_sync(0xffffffffu, sum, 31);
      s_dt[2 * lane] = dt_next[0]; s_dt[2 * lane + 1] = dt_next[1];
      s_L[2 * lane] = sum - e1; s_L[2 * lane + 1] = sum;
      s_w[2 * lane] = exp2f(last - (sum - e1)) * dt_next[0];
      s_w[2 * lane + 1] = exp2f(last - sum) * dt_next[1];
    }
    float2 gate[LOCAL ? 1 : 4][2][2];                            // raw gates of this lane's outputs: requested ahead of the products
    if (!LOCAL && VEC)
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int e = 0; e < 2; ++e)
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const int t = t0 + 16 * i + g4 + 8 * e, c = 16 * warp + 8 * j + l2;
            if (t < t_hi && c < nv) gate[LOCAL ? 0 : i][e][j] = gate2(proj, r0 + t, kx + c);
          }
    if (t0 + CH < t_hi) { fetch(t0 + CH, buf ^ 1); cp_async_wait<1>(); } else cp_async_wait<0>();
    __syncthreads();
    const bf16 *Q = sQ + buf * CH * LQ, *K = sK + buf * CH * LQ, *V = sV + buf * CH * LV;
    if (!LOCAL) {
      // decayed scores of rows 16 warp .. 16 warp + 15
      {
        float p[8][4];
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) p[j][e] = 0.f;
#pragma unroll
        for (int k = 0; k < DT / 16; ++k) {
          unsigned af[4];
          ldmatrix_x4(af[0], af[1], af[2], af[3], Q + (16 * warp + (lane & 15)) * LQ + 16 * k + ((lane >> 4) << 3));
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            if (j > warp) continue;
            unsigned b0[2], b1[2];
            ldmatrix_x4(b0[0], b0[1], b1[0], b1[1], K + (16 * j + (lane & 7) + ((lane >> 4) << 3)) * LQ + 16 * k + (((lane >> 3) & 1) << 3));
            mma_bf16(p[2 * j], af, b0);
            mma_bf16(p[2 * j + 1], af, b1);
          }
        }
        const float Li[2] = {s_L[16 * warp + g4], s_L[16 * warp + g4 + 8]};
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          if (j > 2 * warp + 1) continue;
          const int c = 8 * j + l2;
          const float2 Lj = *reinterpret_cast<const float2*>(s_L + c), dj = *reinterpret_cast<const float2*>(s_dt + c);
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int i = 16 * warp + g4 + 8 * e;
            const float w0 = c <= i ? exp2f(Li[e] - Lj.x) * dj.x : 0.f, w1 = c + 1 <= i ? exp2f(Li[e] - Lj.y) * dj.y : 0.f;
            *reinterpret_cast<float2*>(sP + i * LP + c) = make_float2(p[j][2 * e] * w0, p[j][2 * e + 1] * w1);
          }
        }
      }
      // C S, then the rows' decay
      float o[4][2][4];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) o[i][j][e] = 0.f;
      if (start + t0 > 0) {
#pragma unroll
        for (int k = 0; k < DT / 16; ++k) {
          unsigned b0[2][PIECES], b1[2][PIECES];
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            split2(St[2 * k][2 * e], St[2 * k][2 * e + 1], b0[e]);
            split2(St[2 * k + 1][2 * e], St[2 * k + 1][2 * e + 1], b1[e]);
          }
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            unsigned af[4];
            ldmatrix_x4(af[0], af[1], af[2], af[3], Q + (16 * i + (lane & 15)) * LQ + 16 * k + ((lane >> 4) << 3));
#pragma unroll
            for (int e = 0; e < 2; ++e)
#pragma unroll
              for (int x = PIECES - 1; x >= 0; --x) {
                const unsigned b[2] = {b0[e][x], b1[e][x]};
                mma_bf16(o[i][e], af, b);
              }
          }
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float w0 = exp2f(s_L[16 * i + g4]), w1 = exp2f(s_L[16 * i + g4 + 8]);
#pragma unroll
          for (int e = 0; e < 2; ++e) { o[i][e][0] *= w0; o[i][e][1] *= w0; o[i][e][2] *= w1; o[i][e][3] *= w1; }
        }
      }
      __syncthreads();                                           // scores of all rows are there
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        unsigned b0[2], b1[2];
        ldmatrix_x4_t(b0[0], b0[1], b1[0], b1[1], V + (16 * k + (lane & 7) + (((lane >> 3) & 1) << 3)) * LV + 16 * warp + ((lane >> 4) << 3));
#pragma unroll
        for (int i = k; i < 4; ++i) {
          unsigned ap[4][PIECES];
#pragma unroll
          for (int x = 0; x < 4; ++x) {
            const float2 f = *reinterpret_cast<const float2*>(sP + (16 * i + g4 + 8 * (x & 1)) * LP + 16 * k + l2 + 8 * (x >> 1));
            split2(f.x, f.y, ap[x]);
          }
#pragma unroll
          for (int x = PIECES - 1; x >= 0; --x) {
            const unsigned af[4] = {ap[0][x], ap[1][x], ap[2][x], ap[3][x]};
            mma_bf16(o[i][0], af, b0);
            mma_bf16(o[i][1], af, b1);
          }
        }
      }
      // (y + D x) silu(z)
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int t = 16 * i + g4 + 8 * e;
          if (t >= m) continue;
          const long long row = r0 + t0 + t;
          bf16* out = reinterpret_cast<bf16*>(a.u) + row * inner + kx;
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const int c = 16 * warp + 8 * j + l2;
            if (c >= nv) continue;
            const float2 xv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(V + t * LV + c));
            const float y0 = fmaf(D, xv.x, o[i][j][2 * e]), y1 = fmaf(D, xv.y, o[i][j][2 * e + 1]);
            if (VEC) {
              const float2 z = gate[LOCAL ? 0 : i][e][j];
              *reinterpret_cast<__nv_bfloat162*>(out + c) = __floats2bfloat162_rn(y0 * silu_as<bf16>(z.x), y1 * silu_as<bf16>(z.y));
            } else {
              out[c] = __float2bfloat16_rn(y0 * silu_as<bf16>(proj.get_rare(row, kx + c)));
              if (c + 1 < nv) out[c + 1] = __float2bfloat16_rn(y1 * silu_as<bf16>(proj.get_rare(row, kx + c + 1)));
            }
          }
        }
    }
    // the state behind the chunk
    {
      const float all = exp2f(s_L[CH - 1]);
      total += s_L[CH - 1];
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) St[j][e] *= all;
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        unsigned ar[4], ap[4][PIECES];
        ldmatrix_x4_t(ar[0], ar[1], ar[2], ar[3], V + (16 * k + (lane & 7) + ((lane >> 4) << 3)) * LV + 16 * warp + (((lane >> 3) & 1) << 3));
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&ar[x]));
          const float2 w = *reinterpret_cast<const float2*>(s_w + 16 * k + l2 + 8 * (x >> 1));
          split2(f.x * w.x, f.y * w.y, ap[x]);
        }
#pragma unroll
        for (int j = 0; j < DT / 16; ++j) {
          unsigned b0[2], b1[2];
          ldmatrix_x4_t(b0[0], b0[1], b1[0], b1[1], K + (16 * k + (lane & 7) + (((lane >> 3) & 1) << 3)) * LQ + 16 * j + ((lane >> 4) << 3));
#pragma unroll
          for (int x = PIECES - 1; x >= 0; --x) {
            const unsigned af[4] = {ap[0][x], ap[1][x], ap[2][x], ap[3][x]};
            mma_bf16(St[2 * j], af, b0);
            mma_bf16(St[2 * j + 1], af, b1);
          }
        }
      }
    }
    __syncthreads();
  }
  if (LOCAL && cb == 0 && tid == 0) piece_decay(seg) = total;
  if (!LOCAL && t_hi < n) return;                                // only the last piece ends with the entry's state
  store_state(LOCAL ? piece(seg) : a.state + (((long long)slot * a.R + (start + n) % a.R) * a.H + h) * one);
}

template <int DT, bool VEC, typename S>
int32_t launch_chunks(vn_ctx* ctx, const S& proj, const SsdArgs& a) {
  static unsigned long long done = 0;
  if (!((done >> (ctx->device & 63)) & 1ull)) {
    VN_CUDA(ctx, cudaFuncSetAttribute((ssd_chunk_kernel<DT, false, VEC, S>), cudaFuncAttributeMaxDynamicSharedMemorySize, chunk_smem<DT>(false)));
    VN_CUDA(ctx, cudaFuncSetAttribute((ssd_chunk_kernel<DT, true, VEC, S>), cudaFuncAttributeMaxDynamicSharedMemorySize, chunk_smem<DT>(true)));
    done |= 1ull << (ctx->device & 63);
  }
  const int gx = a.H * ceil_div(a.P, VB);
  if (a.segments > 1)
    VN_LAUNCH_NAMED(ctx, "ssd_segment_kernel", (ssd_chunk_kernel<DT, true, VEC, S>), dim3(gx, a.segments - 1, a.rows.n_ent), 32 * CW,
                    chunk_smem<DT>(true), a, proj);
  VN_LAUNCH_NAMED(ctx, "ssd_chunk_kernel", (ssd_chunk_kernel<DT, false, VEC, S>), dim3(gx, a.segments, a.rows.n_ent), 32 * CW,
                  chunk_smem<DT>(false), a, proj);
  return VN_OK;
}

// ---- norm ------------------------------------------------------------------------------------------------------------------
// One CTA per (part, row); VEC: four columns per thread, NV times (part <= 1024 NV), held between the two passes
template <typename T, int NV>
__global__ void __launch_bounds__(256) ssd_norm_kernel(const T* __restrict__ u, const float* __restrict__ w, T* __restrict__ out, int n,
                                                       int part, float eps) {
  __shared__ float sm[8];
  const int c0 = blockIdx.x * part;
  const long long at = (long long)blockIdx.y * n + c0;
  float ss = 0.f;
  if constexpr (NV > 0) {
    float4 v[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (threadIdx.x + 256 * i) * 4;
      v[i] = c < part ? load4(u + at + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
    const float r = 1.f / sqrtf(block_sum256(ss, sm) / (float)part + eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (threadIdx.x + 256 * i) * 4;
      if (c >= part) break;
      const float4 x = load4(w + c0 + c);
      store4(out + at + c, make_float4(v[i].x * r * x.x, v[i].y * r * x.y, v[i].z * r * x.z, v[i].w * r * x.w));
    }
  } else {
    for (int c = threadIdx.x; c < part; c += 256) { const float v = to_f<T>(u[at + c]); ss += v * v; }
    const float r = 1.f / sqrtf(block_sum256(ss, sm) / (float)part + eps);
    for (int c = threadIdx.x; c < part; c += 256) out[at + c] = from_f<T>(to_f<T>(u[at + c]) * r * w[c0 + c]);
  }
}

}  // namespace

SsdPlan vn_ssd_plan(const vn_ctx* ctx, bool bf16, int H, int N, int P, const Rows& rows, int pending) {
  SsdPlan p;
  // few rows go token by token; so do rows that may be cut back (every state is kept), which only uniform batches have
  p.chunked = bf16 && N <= 128 && rows.max_n >= 8 && rows.max_n > pending;
  if (!p.chunked) return p;
  const long long ctas = (long long)H * ceil_div(P, VB) * rows.n_ent;
  int s = (int)std::min<long long>(8, 2 * ctx->sm_count / std::max(1ll, ctas));
  s = std::max(1, std::min(s, rows.max_n / (4 * CH)));
  p.seg_len = ceil_div(ceil_div(rows.max_n, s), CH) * CH;
  p.segments = ceil_div(rows.max_n, p.seg_len);
  if (p.segments > 1) p.seg_bytes = (size_t)rows.n_ent * p.segments * H * ((size_t)N * P + 1) * 4;
  return p;
}

template <typename T, typename S>
int32_t vn_ssd_inputs(vn_ctx* ctx, const ConvIn<T, S>& conv, const SsdArgs& a) {
  const int M = a.rows.M;
  if constexpr (std::is_same<S, Mat<T>>::value) {
    if (conv.taps <= 4 && conv.C % 4 == 0 && conv.col0 % 4 == 0 && conv.src.ld % 4 == 0 && a.ld % 4 == 0) {
      const int rep = M >= 4096 ? 8 : 2;
      VN_LAUNCH_NAMED(ctx, "ssd_inputs_kernel", (ssd_inputs4_kernel<T, 4>), dim3(ceil_div(conv.C / 4 + a.H, 256), ceil_div(M, 4 * rep)), 256, 0, conv, a, rep);
      return VN_OK;
    }
  }
  const int gx = ceil_div(conv.C, 32) + ceil_div(a.H, 32) + (a.z ? ceil_div(a.inner(), 32) : 0);
  if (M >= 64 && a.rows.max_n > 4)
    VN_LAUNCH_NAMED(ctx, "ssd_inputs_kernel", (ssd_inputs_kernel<T, S, 8>), dim3(gx, ceil_div(M, 64)), dim3(32, 8), 0, conv, a);
  else
    VN_LAUNCH_NAMED(ctx, "ssd_inputs_kernel", (ssd_inputs_kernel<T, S, 1>), dim3(gx, ceil_div(M, 8)), dim3(32, 8), 0, conv, a);
  return VN_OK;
}
template int32_t vn_ssd_inputs(vn_ctx*, const ConvIn<float, Src>&, const SsdArgs&);
template int32_t vn_ssd_inputs(vn_ctx*, const ConvIn<bf16, Src>&, const SsdArgs&);
template int32_t vn_ssd_inputs(vn_ctx*, const ConvIn<bf16, Mat<bf16>>&, const SsdArgs&);

template <typename T, typename S>
int32_t vn_ssd_scan(vn_ctx* ctx, const S& proj, const SsdArgs& a) {
  if (a.rows.max_n == 1 && (a.z || std::is_same<S, Mat<T>>::value) && a.N <= 128 && a.N % 4 == 0 && a.inner() % 4 == 0 && a.ld % 4 == 0) {
    const int np = a.P > SCAN_COLS ? 2 : 1, nb = ceil_div(a.P, SCAN_COLS * np);
    int heads = 8;                                       // as many as leave enough CTAs
    while (heads > 1 && (long long)ceil_div(a.H, heads) * nb * a.rows.n_ent < 3 * ctx->sm_count) heads /= 2;
    const dim3 grid(ceil_div(a.H, heads) * nb, a.rows.n_ent);
    Mat<T> z;
    z.p = (const T*)a.z; z.ld = a.inner();
    if constexpr (std::is_same<S, Mat<T>>::value) z = proj;
#define TOKEN(DK, NP) VN_LAUNCH_NAMED(ctx, "ssd_token_kernel", (ssd_token_kernel<T, DK, NP>), grid, SCAN_TH, 0, a, z, heads)
#define TOKENS(DK) do { if (np == 2) TOKEN(DK, 2); else TOKEN(DK, 1); } while (0)
    if (a.N <= 32) TOKENS(4); else if (a.N <= 64) TOKENS(8); else TOKENS(16);
#undef TOKENS
#undef TOKEN
    return VN_OK;
  }
  ConvIn<T, S> in;
  in.src = proj;
  return launch_scan<T, S, false>(ctx, in, a);
}
template int32_t vn_ssd_scan<float, Src>(vn_ctx*, const Src&, const SsdArgs&);
template int32_t vn_ssd_scan<bf16, Src>(vn_ctx*, const Src&, const SsdArgs&);
template int32_t vn_ssd_scan<bf16, Mat<bf16>>(vn_ctx*, const Mat<bf16>&, const SsdArgs&);

template <typename T>
int32_t vn_ssd_step(vn_ctx* ctx, const ConvIn<T>& conv, const SsdArgs& a) {
  return launch_scan<T, Src, true>(ctx, conv, a);
}
template int32_t vn_ssd_step(vn_ctx*, const ConvIn<float>&, const SsdArgs&);
template int32_t vn_ssd_step(vn_ctx*, const ConvIn<bf16>&, const SsdArgs&);

template <typename S>
int32_t vn_ssd_chunks(vn_ctx* ctx, const S& proj, const SsdArgs& a) {
  const bool vec = a.N % 8 == 0 && a.P % 8 == 0 && a.ld % 8 == 0 && proj.ld % 2 == 0;
#define CHUNKS(DT) return vec ? launch_chunks<DT, true>(ctx, proj, a) : launch_chunks<DT, false>(ctx, proj, a)
  if (a.N <= 32) CHUNKS(32);
  if (a.N <= 64) CHUNKS(64);
  if (a.N <= 128) CHUNKS(128);
#undef CHUNKS
  return vn_fail(ctx, VN_ERR_UNSUPPORTED, "state size %d", a.N);
}
template int32_t vn_ssd_chunks(vn_ctx*, const Src&, const SsdArgs&);
template int32_t vn_ssd_chunks(vn_ctx*, const Mat<bf16>&, const SsdArgs&);

template <typename T>
int32_t vn_ssd_norm(vn_ctx* ctx, const T* u, const float* w, T* out, int M, int n, int parts, float eps) {
  const int part = n / parts;
  const dim3 grid(parts, M);
#define NORM(NV) VN_LAUNCH_NAMED(ctx, "ssd_norm_kernel", (ssd_norm_kernel<T, NV>), grid, 256, 0, u, w, out, n, part, eps)
  if (part % 4 || part > 8192) NORM(0); else if (part <= 1024) NORM(1); else if (part <= 4096) NORM(4); else NORM(8);
#undef NORM
  return VN_OK;
}
template int32_t vn_ssd_norm(vn_ctx*, const float*, const float*, float*, int, int, int, float);
template int32_t vn_ssd_norm(vn_ctx*, const bf16*, const float*, bf16*, int, int, int, float);
