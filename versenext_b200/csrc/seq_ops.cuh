// Kernels shared by the layer kinds of composed models (hybrid.cuh): embedding with position vectors, the entry of a
// looped block, row sums with a norm, the end of a sublayer, activations of feed-forwards, picked rows, and the tail of the
// convolution inputs.
#pragma once
#include "model_kernels.cuh"

// ---- token embedding + sinusoidal position vector: entry 2i sin, 2i+1 cos of pos * freq[i]; x and a copy x0 (or null).
// The angle is reduced to one turn in double before the float sine, so far positions lose nothing.
template <typename T>
__global__ void __launch_bounds__(256) embed_pos_kernel(const long long* __restrict__ tokens, const T* __restrict__ emb,
                                                        const double* __restrict__ freq, float* __restrict__ x,
                                                        float* __restrict__ x0, Rows rows, int D, int V,
                                                        int* __restrict__ status) {
  const int row = blockIdx.x;
  long long tok = tokens[row];
  if (tok < 0 || tok >= V) {
    if (threadIdx.x == 0) atomicExch(status, 1);
    tok = tok < 0 ? 0 : V - 1;
  }
  int slot, r0, n, start;
  rows.entry(rows.entry_of(row), &slot, &r0, &n, &start);
  const int pos = start + row - r0;
  const T* e = emb + tok * D;
  for (int i = threadIdx.x; 2 * i < D; i += 256) {
    float sn = 0.f, cs = 0.f;
    if (freq) {
      const double a = (double)pos * freq[i];
      const double turn = 6.283185307179586476925;
      const float r = (float)(a - rint(a / turn) * turn);
      sincosf(r, &sn, &cs);
    }
    const long long o = (long long)row * D + 2 * i;
    const float v0 = to_f<T>(e[2 * i]) + sn;
    x[o] = v0;
    if (x0) x0[o] = v0;
    if (2 * i + 1 < D) {
      const float v1 = to_f<T>(e[2 * i + 1]) + cs;
      x[o + 1] = v1;
      if (x0) x0[o + 1] = v1;
    }
  }
}

// operand of a pass's entry projection: [x | x0] in the storage dtype
template <typename T>
__global__ void __launch_bounds__(256) concat_cast_kernel(const float* __restrict__ x, const float* __restrict__ x0,
                                                          T* __restrict__ out, int D) {
  const long long row = blockIdx.x;
  for (int d = threadIdx.x; d < D; d += 256) {
    out[row * 2 * D + d] = from_f<T>(x[row * D + d]);
    out[row * 2 * D + D + d] = from_f<T>(x0[row * D + d]);
  }
}

// x = (keep ? x : 0) + sum of slices (+ bias); then, if norm_w, y = RMSNorm(x) * norm_w.  Any D.
template <typename T>
__global__ void __launch_bounds__(256) rowsum_norm_kernel(Src src, const float* __restrict__ bias, int keep,
                                                          float* __restrict__ x, const float* __restrict__ norm_w,
                                                          T* __restrict__ y, int D, float eps) {
  __shared__ float sm[8];
  const long long row = blockIdx.x;
  float ss = 0.f;
  for (int d = threadIdx.x; d < D; d += 256) {
    float v = src.get(row, d);
    if (bias) v += bias[d];
    if (keep) v += x[row * D + d];
    x[row * D + d] = v;
    ss += v * v;
  }
  if (!norm_w) return;
  const float r = sqrtf(block_sum256(ss, sm) / (float)D + eps);
  for (int d = threadIdx.x; d < D; d += 256) y[row * D + d] = from_f<T>(x[row * D + d] / r * norm_w[d]);
}

// Entry of a looped block that adds instead of projecting: x += x0 (from the second pass on) + step vector of the pass.
struct PassEntry { const float* x0 = nullptr; const float* step = nullptr; };

// the same by itself, with the norm of the pass's first layer behind it.  Any D, grid M
template <typename T>
__global__ void __launch_bounds__(256) enter_pass_kernel(PassEntry pass, float* __restrict__ x, const float* __restrict__ norm_w,
                                                         T* __restrict__ y, int D, float eps) {
  __shared__ float sm[8];
  const long long row = blockIdx.x;
  float ss = 0.f;
  for (int d = threadIdx.x; d < D; d += 256) {
    float v = x[row * D + d];
    if (pass.x0) v += pass.x0[row * D + d];
    v += pass.step[d];
    x[row * D + d] = v;
    ss += v * v;
  }
  const float r = sqrtf(block_sum256(ss, sm) / (float)D + eps);
  for (int d = threadIdx.x; d < D; d += 256) y[row * D + d] = from_f<T>(x[row * D + d] / r * norm_w[d]);
}

// ---- the end of a sublayer in one pass over a row: what it adds, the residual, and what the next product reads -------------
// Y gives the addend: quad(row, d) of four columns, one(row, d) of one; begin(row) is called by all 256 threads first.

// a projection's result with a bias
template <typename S>
struct AddRows {
  S y;
  const float* bias = nullptr;
  __device__ __forceinline__ void begin(int) {}
  __device__ __forceinline__ float4 quad(int row, int d) const {
    float4 v = get4(y, row, d);
    if (bias) { const float4 b = load4(bias + d); v.x += b.x; v.y += b.y; v.z += b.z; v.w += b.w; }
    return v;
  }
  __device__ __forceinline__ float one(int row, int d) const { return y.get(row, d) + (bias ? bias[d] : 0.f); }
};

// the results of a row's experts: rows slot_pos[] of y, weighted unless the weights are null; experts from n_real on are the
// input h itself; and the gated result of the expert that serves every row, a matrix of its own or that of a row's last slot
template <typename T, typename S>
struct AddExperts {
  S y;
  const T* h = nullptr;
  const int *slot_pos = nullptr, *slot_expert = nullptr;
  const float* slot_w = nullptr;
  S shared;                                      // [M, D], times shared_gate [M] (null: none)
  const float* shared_gate = nullptr;
  const float* slot_gate = nullptr;              // [M] factor of slot top - 1, or null
  int top = 1, n_real = 0, D = 0;
  int *count = nullptr, *cursor = nullptr;       // left at zero for the next mixture
  int n_count = 0;
  int* pos;                                      // of the chosen experts with results; shared memory
  float* w;
  int n;
  float w_self;
  __device__ __forceinline__ void begin(int row) {
    __shared__ int s_pos[32];
    __shared__ float s_w[32];
    pos = s_pos; w = s_w;
    const int lane = threadIdx.x & 31;           // every warp finds out for itself; they write the same values
    const bool has = lane < top;
    const int e = has ? slot_expert[(long long)row * top + lane] : n_real;
    const float v = !has ? 0.f : slot_gate && lane == top - 1 ? slot_gate[row] : slot_w ? slot_w[(long long)row * top + lane] : 1.f;
    const unsigned real = __ballot_sync(0xffffffffu, has && e < n_real);
    if (has && e < n_real) {
      const int at = __popc(real & ((1u << lane) - 1));
      s_pos[at] = slot_pos[(long long)row * top + lane];
      s_w[at] = v;
    }
    n = __popc(real);
    w_self = warp_sum(has && e >= n_real ? v : 0.f);
    if (blockIdx.x == 0)
      for (int i = threadIdx.x; i < n_count; i += 256) { count[i] = 0; cursor[i] = 0; }
    __syncthreads();
  }
  __device__ __forceinline__ float4 quad(int row, int d) const {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    if (shared_gate) a = scaled(get4(shared, row, d), shared_gate[row]);
    if (w_self != 0.f) { const float4 t = load4(h + (long long)row * D + d); a = make_float4(fmaf(t.x, w_self, a.x), fmaf(t.y, w_self, a.y), fmaf(t.z, w_self, a.z), fmaf(t.w, w_self, a.w)); }
#pragma unroll 4
    for (int j = 0; j < n; ++j) {
      const float4 t = get4(y, pos[j], d);
      const float f = w[j];
      a.x = fmaf(t.x, f, a.x); a.y = fmaf(t.y, f, a.y); a.z = fmaf(t.z, f, a.z); a.w = fmaf(t.w, f, a.w);
    }
    return a;
  }
  __device__ __forceinline__ float one(int row, int d) const {
    float a = w_self != 0.f ? w_self * to_f<T>(h[(long long)row * D + d]) : 0.f;
    if (shared_gate) a = fmaf(shared.get(row, d), shared_gate[row], a);
    for (int j = 0; j < n; ++j) a = fmaf(y.get(pos[j], d), w[j], a);
    return a;
  }
};

// x += y, or y over its root mean square times own_norm, and what a pass of a looped block begins with; then h = RMSNorm(x) * next_norm, or x itself (cast), or nothing.
// NV > 0: four columns per thread, NV times, held in registers (D % 4 == 0, D <= 1024 NV); 0: any D.  grid M
template <typename T, typename Y, int NV>
__global__ void __launch_bounds__(256) residual_kernel(Y y, float* __restrict__ x, const float* __restrict__ own_norm,
                                                       PassEntry pass, const float* __restrict__ next_norm, int cast, T* __restrict__ h, int D, float eps) {
  __shared__ float sm[2][8];
  pdl_trigger();
  pdl_wait();
  const int row = blockIdx.x;
  float* xr = x + (long long)row * D;
  T* hr = h + (long long)row * D;
  y.begin(row);
  float ss = 0.f;
  if constexpr (NV > 0) {
    float4 v[NV], xv[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int d = (threadIdx.x + 256 * i) * 4;
      v[i] = xv[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (d < D) { xv[i] = load4(xr + d); v[i] = y.quad(row, d); }
    }
    if (own_norm) {
#pragma unroll
      for (int i = 0; i < NV; ++i) ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
      const float r = 1.f / sqrtf(block_sum256(ss, sm[0]) / (float)D + eps);
      ss = 0.f;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int d = (threadIdx.x + 256 * i) * 4;
        if (d >= D) break;
        const float4 w = load4(own_norm + d);
        v[i] = make_float4(v[i].x * r * w.x, v[i].y * r * w.y, v[i].z * r * w.z, v[i].w * r * w.w);
      }
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int d = (threadIdx.x + 256 * i) * 4;
      if (d >= D) break;
      xv[i] = make_float4(xv[i].x + v[i].x, xv[i].y + v[i].y, xv[i].z + v[i].z, xv[i].w + v[i].w);
      if (pass.step) {
        if (pass.x0) { const float4 t = load4(pass.x0 + (long long)row * D + d); xv[i] = make_float4(xv[i].x + t.x, xv[i].y + t.y, xv[i].z + t.z, xv[i].w + t.w); }
        const float4 t = load4(pass.step + d);
        xv[i] = make_float4(xv[i].x + t.x, xv[i].y + t.y, xv[i].z + t.z, xv[i].w + t.w);
      }
      store4(xr + d, xv[i]);
      if (cast) store4(hr + d, xv[i]);
      ss += xv[i].x * xv[i].x + xv[i].y * xv[i].y + xv[i].z * xv[i].z + xv[i].w * xv[i].w;
    }
    if (!next_norm) return;
    const float r = 1.f / sqrtf(block_sum256(ss, sm[1]) / (float)D + eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int d = (threadIdx.x + 256 * i) * 4;
      if (d >= D) break;
      const float4 w = load4(next_norm + d);
      store4(hr + d, make_float4(xv[i].x * r * w.x, xv[i].y * r * w.y, xv[i].z * r * w.z, xv[i].w * r * w.w));
    }
  } else {
    float f = 1.f;
    if (own_norm) {
      for (int d = threadIdx.x; d < D; d += 256) { const float v = y.one(row, d); ss += v * v; }
      f = 1.f / sqrtf(block_sum256(ss, sm[0]) / (float)D + eps);
      ss = 0.f;
    }
    for (int d = threadIdx.x; d < D; d += 256) {
      float v = y.one(row, d);
      if (own_norm) v *= f * own_norm[d];
      v += xr[d];
      if (pass.x0) v += pass.x0[(long long)row * D + d];
      if (pass.step) v += pass.step[d];
      xr[d] = v;
      if (cast) hr[d] = from_f<T>(v);
      ss += v * v;
    }
    if (!next_norm) return;
    const float r = 1.f / sqrtf(block_sum256(ss, sm[1]) / (float)D + eps);
    for (int d = threadIdx.x; d < D; d += 256) hr[d] = from_f<T>(xr[d] * r * next_norm[d]);
  }
}

// A layer's own input for a token: act = gelu(gate) * the layer's part of the token's side embedding, n columns padded to ld.
// table [V, pitch]; grid ceil(M ld / 256)
template <typename T>
__global__ void __launch_bounds__(256) side_act_kernel(Src gate, const long long* __restrict__ tokens, int V, const T* __restrict__ table,
                                                       long long pitch, int col0, int n, T* __restrict__ act, int ld, long long total) {
  pdl_trigger();
  pdl_wait();
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i >= total) return;
  const long long row = i / ld;
  const int j = (int)(i % ld);
  long long tok = tokens[row];
  tok = tok < 0 ? 0 : tok >= V ? V - 1 : tok;            // the embedding has raised the flag
  act[i] = from_f<T>(j < n ? gelu_tanh(gate.get(row, j)) * to_f<T>(table[tok * pitch + col0 + j]) : 0.f);
}

// PolyNorm: act = a N(z) + b N(z^2) + c N(z^3) + e over a row of n columns, N: over the root mean square; coef = {a, b, c, e}.
// Columns n .. ld - 1 of z are zero (and meet zero weights behind).  NV > 0: four columns per thread, NV times, held in
// registers (ld % 4 == 0, ld <= 1024 NV); 0: any ld, z is read twice.  grid M
template <typename T, typename S, int NV>
__global__ void __launch_bounds__(256) poly_norm_kernel(S z, const float* __restrict__ coef, T* __restrict__ act, int n, int ld, float eps) {
  __shared__ float sm[3][8];
  pdl_trigger();
  pdl_wait();
  const int row = blockIdx.x;
  T* out = act + (long long)row * ld;
  float s2 = 0.f, s4 = 0.f, s6 = 0.f;
  auto count = [&](float v) { const float q = v * v; s2 += q; s4 = fmaf(q, q, s4); s6 = fmaf(q * q, q, s6); };
  float4 v[NV > 0 ? NV : 1];
  if constexpr (NV > 0) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (threadIdx.x + 256 * i) * 4;
      v[i] = c < ld ? get4(z, row, c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) { count(v[i].x); count(v[i].y); count(v[i].z); count(v[i].w); }
  } else {
    for (int c = threadIdx.x; c < n; c += 256) count(z.get(row, c));
  }
  s2 = warp_sum(s2); s4 = warp_sum(s4); s6 = warp_sum(s6);
  if ((threadIdx.x & 31) == 0) { const int w = threadIdx.x >> 5; sm[0][w] = s2; sm[1][w] = s4; sm[2][w] = s6; }
  __syncthreads();
  float f[3];
#pragma unroll
  for (int k = 0; k < 3; ++k) {
    float t = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) t += sm[k][w];
    f[k] = coef[k] / sqrtf(t / (float)n + eps);
  }
  const float e = coef[3];
  auto value = [&](float x) { return fmaf(x, fmaf(x, fmaf(x, f[2], f[1]), f[0]), e); };
  if constexpr (NV > 0) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (threadIdx.x + 256 * i) * 4;
      if (c < ld) store4(out + c, make_float4(value(v[i].x), value(v[i].y), value(v[i].z), value(v[i].w)));
    }
  } else {
    for (int c = threadIdx.x; c < ld; c += 256) out[c] = from_f<T>(value(c < n ? z.get(row, c) : 0.f));
  }
}

// y = RMSNorm(x[row_of(i)]) * w: rows picked by a list, by (i * mul + add), or the entries' last rows
template <typename T>
__global__ void __launch_bounds__(256) rmsnorm_pick_kernel(const float* __restrict__ x, const float* __restrict__ w,
                                                           T* __restrict__ y, float* __restrict__ y32,
                                                           const int* __restrict__ pick, int mul, int add, int D, float eps) {
  __shared__ float sm[8];
  const long long src = pick ? pick[blockIdx.x] : (long long)blockIdx.x * mul + add;
  const float* xr = x + src * D;
  float ss = 0.f;
  for (int d = threadIdx.x; d < D; d += 256) ss += xr[d] * xr[d];
  const float r = sqrtf(block_sum256(ss, sm) / (float)D + eps);
  for (int d = threadIdx.x; d < D; d += 256) {
    const float v = xr[d] / r * w[d];
    if (y) y[(long long)blockIdx.x * D + d] = from_f<T>(v);
    if (y32) y32[(long long)blockIdx.x * D + d] = v;
  }
}

// sum of split-K slices [M, N]: columns below n_act through a function (GemmPost) to `act` [M, ld_act] in the storage dtype,
// the others as they are to `rest` [M, N - n_act] in fp32 (or, with rest null, to `act` too).  N % 4 == n_act % 4 == 0.
template <typename T>
__global__ void __launch_bounds__(256) slices_act_kernel(Src src, int N, int n_act, int post, T* __restrict__ act, int ld_act,
                                                         float* __restrict__ rest, long long total4) {
  pdl_trigger();
  pdl_wait();
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i >= total4) return;
  const long long row = i / (N / 4);
  const int c = (int)(i % (N / 4)) * 4;
  float4 v = get4(src, row, c);
  if (c >= n_act && rest) {
    store4(rest + row * (N - n_act) + c - n_act, v);
    return;
  }
  if (c < n_act) {
    constexpr bool fast = sizeof(T) == 2;
    v = make_float4(post_act(v.x, post, fast), post_act(v.y, post, fast), post_act(v.z, post, fast), post_act(v.w, post, fast));
  }
  store4(act + row * ld_act + c, v);
}
// the same one column at a time: columns [0, N) of the source's rows to a matrix [M, N], any sizes
template <typename T>
__global__ void __launch_bounds__(256) slices_act1_kernel(Src src, int N, int n_act, int post, T* __restrict__ act, long long total) {
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i >= total) return;
  const int c = (int)(i % N);
  const float v = src.get(i / N, c);
  act[i] = from_f<T>(c < n_act ? post_act(v, post, sizeof(T) == 2) : v);
}

// lens[slot] += rows of the entry (a step that keeps everything it appended)
__global__ void rows_advance_kernel(Rows rows, int* __restrict__ lens) {
  const int e = blockIdx.x * blockDim.x + threadIdx.x;
  if (e >= rows.n_ent) return;
  lens[rows.T > 0 ? rows.slot0 + e : rows.slot[e]] += rows.T > 0 ? rows.T : rows.cnt[e];
}

// inputs of long entries (more rows than the ring keeps apart): the last taps - 1 positions, after every reader of
// the older ones has finished.  grid (ceil(C / 256), n_ent)
template <typename T, typename S, bool ACT>
__global__ void __launch_bounds__(256) conv_tail_kernel(ConvIn<T, S, ACT> in, Rows rows, int pending) {
  int slot, r0, n, start;
  rows.entry(blockIdx.y, &slot, &r0, &n, &start);
  const int c = blockIdx.x * 256 + threadIdx.x;
  if (n <= pending || c >= in.C) return;
  const int first = max(0, n - (in.taps - 1));
  for (int t = first; t < n; ++t) in.keep(slot, start + t, c, in.src.get(r0 + t, in.col0 + c));
}
