// Device-side vocabulary of the row kernels: storage-type conversion, where a row of a (ragged) batch sits in its
// sequence, sums over split-K slices, and the short causal convolution with its cached inputs.  No kernels here: the file
// is included by several translation units.
#pragma once
#include "common.cuh"

template <typename T> __device__ __forceinline__ float to_f(T v);
template <> __device__ __forceinline__ float to_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

constexpr int KV_PAGE = 64;      // tokens of a cache page

// Rows of a forward.  Either a uniform batch (T > 0: entry e = sequence slot0 + e, rows [e*T, e*T + T)) or a ragged
// one (T == 0: tables).  Row r of an entry that starts at row row0 has position lens[slot] + off + (r - row0).
struct Rows {
  int T = 0, slot0 = 0, off = 0, n_ent = 0, M = 0, max_n = 0;
  const int* ent = nullptr;    // [M] entry of a row
  const int* slot = nullptr;   // [n_ent]
  const int* row0 = nullptr;   // [n_ent]
  const int* cnt = nullptr;    // [n_ent]
  const int* lens = nullptr;   // [slots] committed tokens

  __device__ __forceinline__ int entry_of(int row) const { return T > 0 ? row / T : ent[row]; }
  __device__ __forceinline__ void entry(int e, int* s, int* r0, int* n, int* start) const {
    if (T > 0) { *s = slot0 + e; *r0 = e * T; *n = T; }
    else { *s = slot[e]; *r0 = row0[e]; *n = cnt[e]; }
    *start = lens[*s] + off;
  }
};

// sum of split-K slices of one value, out of line: for code that needs many such values on a rare path
static __device__ __noinline__ float sum_slices(const float* q, int splits, long long pstride) {
  float a = 0.f;
  for (int s = 0; s < splits; ++s) a += q[s * pstride];
  return a;
}

// the fp32 result of a projection: one matrix, or split-K slices that the reader sums in slice order
struct Src {
  const float* p = nullptr;
  int splits = 1;
  long long pstride = 0;
  int ld = 0;
  __device__ __forceinline__ float get(long long row, int col) const {
    const float* q = p + row * ld + col;
    if (splits == 1) return *q;
    float a = 0.f;
    int s = 0;
    for (; s + 4 <= splits; s += 4) {          // four slices requested before the first is added; slice order kept
      const float t0 = q[s * pstride], t1 = q[(s + 1) * pstride], t2 = q[(s + 2) * pstride], t3 = q[(s + 3) * pstride];
      a += t0; a += t1; a += t2; a += t3;
    }
    for (; s < splits; ++s) a += q[s * pstride];
    return a;
  }
  __device__ __forceinline__ float get_rare(long long row, int col) const { return sum_slices(p + row * ld + col, splits, pstride); }
  // rows row .. row + RB - 1 of a column (clamped to row_end - 1), loads independent of one another
  template <int RB>
  __device__ __forceinline__ void column(int row, int row_end, int col, float (&out)[RB]) const {
    if (splits == 1) {
      const float* q = p + (long long)row * ld + col;
#pragma unroll
      for (int i = 0; i < RB; ++i) out[i] = q[(long long)(min(row + i, row_end - 1) - row) * ld];
    } else {
#pragma unroll
      for (int i = 0; i < RB; ++i) out[i] = get(min(row + i, row_end - 1), col);
    }
  }
};

// the same as a matrix in the storage dtype (many rows of a 16-bit model: half the bytes)
template <typename T>
struct Mat {
  const T* p = nullptr;
  int ld = 0;
  static constexpr int splits = 1;
  __device__ __forceinline__ float get(long long row, int col) const { return to_f<T>(p[row * ld + col]); }
  __device__ __forceinline__ float get_rare(long long row, int col) const { return get(row, col); }
};

// four neighbouring columns (16-byte aligned fp32, 8-byte aligned 16-bit)
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
  uint2 u;
  *reinterpret_cast<__nv_bfloat162*>(&u.x) = __floats2bfloat162_rn(v.x, v.y);
  *reinterpret_cast<__nv_bfloat162*>(&u.y) = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = u;
}
__device__ __forceinline__ float4 scaled(float4 v, float f) { return make_float4(v.x * f, v.y * f, v.z * f, v.w * f); }
__device__ __forceinline__ float4 get4(const Src& s, long long row, int col) {
  const float* q = s.p + row * s.ld + col;
  float4 a = load4(q);
#pragma unroll 4
  for (int i = 1; i < s.splits; ++i) {
    const float4 t = load4(q + (long long)i * s.pstride);
    a.x += t.x; a.y += t.y; a.z += t.z; a.w += t.w;
  }
  return a;
}
template <typename T>
__device__ __forceinline__ float4 get4(const Mat<T>& s, long long row, int col) { return load4(s.p + row * s.ld + col); }

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
// silu of a value that is kept in T: the fast exponential and division where that is 16 bits wide
template <typename T> __device__ __forceinline__ float silu_as(float z) {
  return sizeof(T) == 2 ? __fdividef(z, 1.0f + __expf(-z)) : z / (1.0f + expf(-z));
}
template <typename T> __device__ __forceinline__ float round_to(float v) { return to_f<T>(from_f<T>(v)); }

// block-wide sum of one value per thread (256 threads), the same total in every thread
__device__ __forceinline__ float block_sum256(float v, float* sm8) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) sm8[threadIdx.x >> 5] = v;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) tot += sm8[i];
  return tot;
}

// ---- short causal convolution over time, one filter per channel ----------------------------------------------
// The inputs of position p of slot s are kept at ring[(s * RC + p % RC) * C]: the last taps - 1 of them are state, the
// others are inputs of positions that are appended and not committed yet (a rejected suffix is simply overwritten).
// An input is rounded to the storage dtype before it is used, so that it does not matter whether it came from this
// forward or from the ring.
// S: where this forward's rows come from.  ACT: silu behind the sum, or nothing.
template <typename T, typename S = Src, bool ACT = true>
struct ConvIn {
  S src;                   // projection rows of this forward
  int col0 = 0;            // first convolved column
  T* ring = nullptr;
  int RC = 1, C = 0, taps = 1;
  const float* w = nullptr;      // [C, taps]
  const float* bias = nullptr;   // [C] or null
  bool named = true;             // false: one tap of weight 1, the inputs themselves

  template <bool RARE = false>
  __device__ __forceinline__ float input(int row, int r0, int start, int slot, int pos, int c) const {
    if (pos >= start) return round_to<T>(RARE ? src.get_rare(r0 + pos - start, col0 + c) : src.get(r0 + pos - start, col0 + c));
    if (pos < 0) return 0.f;
    return to_f<T>(ring[((long long)slot * RC + pos % RC) * C + c]);
  }
  // the activated sum of channel c at `row`; *cur receives the row's own input
  __device__ __forceinline__ float at(int row, int r0, int start, int slot, int c, float* cur) const {
    const int pos = start + row - r0;
    const float* wc = w + (long long)c * taps;
    float acc, x[4], f[4];
    if (taps <= 4) {                           // the usual lengths: all inputs requested before the first is used
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        f[j] = j < taps ? wc[taps - 1 - j] : 0.f;
        x[j] = j < taps ? input(row, r0, start, slot, pos - j, c) : 0.f;
      }
      acc = x[0] * f[0];
#pragma unroll
      for (int j = 1; j < 4; ++j) acc = fmaf(x[j], f[j], acc);
    } else {
      x[0] = input(row, r0, start, slot, pos, c);
      acc = x[0] * wc[taps - 1];
      for (int j = 1; j < taps; ++j) acc = fmaf(input(row, r0, start, slot, pos - j, c), wc[taps - 1 - j], acc);
    }
    *cur = x[0];
    return activate(acc, c);
  }
  __device__ __forceinline__ float activate(float acc, int c) const {
    if (bias) acc += bias[c];
    return ACT ? silu_as<T>(acc) : acc;
  }
  // The same for rows row, row + 1, .. row + RB - 1 (those below row_end, all of one entry): every input is read once.
  // taps <= 4.  Nothing is stored here, so that the loads of several calls can be in flight together.
  template <int RB>
  __device__ __forceinline__ void run(int row, int row_end, int r0, int start, int slot, int c, float (&out)[RB]) const {
    const int pos = start + row - r0;
    const float* wc = w + (long long)c * taps;
    float wt[4], x[RB + 3];
    if (taps == 4) {
      const float4 t = *reinterpret_cast<const float4*>(wc);
      wt[0] = t.w; wt[1] = t.z; wt[2] = t.y; wt[3] = t.x;
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j) wt[j] = j < taps ? wc[taps - 1 - j] : 0.f;
    }
    if (src.splits == 1 && row - r0 >= 3) {            // inside an entry's rows: plain loads, all independent
      const auto* p = src.p + (long long)row * src.ld + col0 + c;
      if (row + RB <= row_end) {
        p -= 3ll * src.ld;
#pragma unroll
        for (int i = 0; i < RB + 3; ++i, p += src.ld) x[i] = to_f(*p);
      } else {
#pragma unroll
        for (int i = 0; i < RB + 3; ++i) x[i] = to_f(p[(long long)(min(row + i - 3, row_end - 1) - row) * src.ld]);
      }
#pragma unroll
      for (int i = 0; i < RB + 3; ++i) x[i] = round_to<T>(x[i]);
    } else {
#pragma unroll
      for (int j = 1; j < 4; ++j) x[3 - j] = j < taps ? input<true>(row, r0, start, slot, pos - j, c) : 0.f;
#pragma unroll
      for (int i = 0; i < RB; ++i) x[3 + i] = row + i < row_end ? round_to<T>(src.get_rare(row + i, col0 + c)) : 0.f;
    }
#pragma unroll
    for (int i = 0; i < RB; ++i) {
      float acc = x[3 + i] * wt[0];
#pragma unroll
      for (int j = 1; j < 4; ++j) acc = fmaf(x[3 + i - j], wt[j], acc);
      out[i] = activate(acc, c);
    }
  }
  // The same for channels c .. c + 3 of a matrix in the storage dtype (col0 + c, the pitch and c multiples of 4).
  // wt: filters4(c), [tap back][channel].
  __device__ __forceinline__ void filters4(int c, float (&wt)[4][4]) const {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float* wc = w + (long long)(c + e) * taps;
      if (taps == 4) {
        const float4 t = *reinterpret_cast<const float4*>(wc);
        wt[0][e] = t.w; wt[1][e] = t.z; wt[2][e] = t.y; wt[3][e] = t.x;
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j) wt[j][e] = j < taps ? wc[taps - 1 - j] : 0.f;
      }
    }
  }
  template <int RB>
  __device__ __forceinline__ void run4(int row, int row_end, int r0, int start, int slot, int c, const float (&wt)[4][4],
                                       float4 (&out)[RB]) const {
    float4 x[RB + 3];
    const auto* p = src.p + (long long)row * src.ld + col0 + c;
#pragma unroll
    for (int i = 0; i < RB; ++i) x[3 + i] = load4(p + (long long)(min(row + i, row_end - 1) - row) * src.ld);
    if (taps == 1) {
#pragma unroll
      for (int i = 0; i < 3; ++i) x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    } else if (row - r0 >= 3) {
#pragma unroll
      for (int i = 0; i < 3; ++i) x[i] = load4(p + (long long)(i - 3) * src.ld);
    } else {
      const int pos = start + row - r0;
#pragma unroll
      for (int j = 1; j < 4; ++j) {
        x[3 - j] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (j < taps)
          x[3 - j] = make_float4(input(row, r0, start, slot, pos - j, c), input(row, r0, start, slot, pos - j, c + 1),
                                 input(row, r0, start, slot, pos - j, c + 2), input(row, r0, start, slot, pos - j, c + 3));
      }
    }
#pragma unroll
    for (int i = 0; i < RB; ++i) {
      float a[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        auto at = [&](const float4& v) { return e == 0 ? v.x : e == 1 ? v.y : e == 2 ? v.z : v.w; };
        a[e] = at(x[3 + i]) * wt[0][e];
#pragma unroll
        for (int j = 1; j < 4; ++j) a[e] = fmaf(at(x[3 + i - j]), wt[j][e], a[e]);
        a[e] = activate(a[e], c + e);
      }
      out[i] = make_float4(a[0], a[1], a[2], a[3]);
    }
  }
  __device__ __forceinline__ void keep(int slot, int pos, int c, float v) const {
    ring[((long long)slot * RC + pos % RC) * C + c] = from_f<T>(v);
  }
};
