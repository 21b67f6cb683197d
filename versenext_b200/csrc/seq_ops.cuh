// Kernels shared by the layer kinds of composed models (hybrid.cuh): embedding with position vectors, the entry of a
// looped block, row sums with a norm, picked rows, and the tail of the convolution inputs.
#pragma once
#include "model_kernels.cuh"

// ---- token embedding + sinusoidal position vector: entry 2i sin, 2i+1 cos of pos * freq[i]; x and a copy x0.
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
    x[o] = v0; x0[o] = v0;
    if (2 * i + 1 < D) {
      const float v1 = to_f<T>(e[2 * i + 1]) + cs;
      x[o + 1] = v1; x0[o + 1] = v1;
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
