// Kernels of paged_attn.cuh for prompts and mixed batches; the one-token kernel is in attn_step.cu.
#include <algorithm>
#include <type_traits>

#include "ldmatrix.cuh"
#include "paged_attn.cuh"

namespace {

using bf16 = __nv_bfloat16;

__global__ void __launch_bounds__(128) rope_table_kernel(const double* __restrict__ freq, int pairs, float amp, long long total,
                                                         float2* __restrict__ out) {
  const long long i = (long long)blockIdx.x * 128 + threadIdx.x;
  if (i >= total) return;
  double s, c;
  sincos((double)(i / pairs) * freq[i % pairs], &s, &c);
  out[i] = make_float2((float)(c * (double)amp), (float)(s * (double)amp));
}

// One warp per (RB rows, unit): units 0 .. H-1 query heads, then KH key heads and KH value heads (own_kv).  A lane takes
// both channels of a rotated pair.  RB > 1: filters of at most four taps.  grid (units, ceil(M / (8 RB))), block (32, 8)
template <typename T, typename S, int RB>
__global__ void __launch_bounds__(256) attn_inputs_kernel(ConvIn<T, S, false> in, PagedAttnArgs a) {
  const int lane = threadIdx.x, unit = blockIdx.x;
  int row = (blockIdx.y * 8 + threadIdx.y) * RB;
  const int last = min(row + RB, a.rows.M);
  const bool is_q = unit < a.H, is_v = unit >= a.H + a.KH;
  const int head = is_q ? unit : is_v ? unit - a.H - a.KH : unit - a.H;
  const int w = is_v ? a.vd : a.d;
  const int c0 = is_v ? (a.H + a.KH) * a.d + head * a.vd : unit * a.d;
  const int np = is_v ? 0 : a.rd / 2, items = w - np;       // pairs first, then single channels
  const float tf = is_q && a.temp ? a.temp[head] : 1.f;
  while (row < last) {                                      // stretches of one entry
    int slot, r0, n, start;
    a.rows.entry(a.rows.entry_of(row), &slot, &r0, &n, &start);
    const int first = row, end = min(last, r0 + n);
    auto convolve = [&](int c, float (&v)[RB]) {
      if constexpr (RB > 1) {
        in.template run<RB>(first, end, r0, start, slot, c0 + c, v);
      } else {
        float cur;
        v[0] = in.at(first, r0, start, slot, c0 + c, &cur);
      }
      if (n <= a.pending && in.taps > 1)
        for (int r = first; r < end; ++r) in.keep(slot, start + r - r0, c0 + c, in.src.get_rare(r, in.col0 + c0 + c));
    };
    auto dest = [&](int r) -> T* {
      if (is_q) return reinterpret_cast<T*>(a.q) + ((long long)r * a.H + head) * a.P;
      const int pos = start + r - r0;
      T* plane = reinterpret_cast<T*>(is_v ? a.vplane : a.kplane);
      return plane + (((long long)a.table[(long long)slot * a.max_pages + pos / KV_PAGE] * KV_PAGE + pos % KV_PAGE) * a.KH + head) * a.P;
    };
    for (int i = lane; i < items; i += 32) {
      const bool pair = i < np;
      const int cu = !pair ? np + i : a.interleaved ? 2 * i : i, cv = a.interleaved ? 2 * i + 1 : np + i;
      float u[RB], v[RB];
      convolve(cu, u);
      if (pair) convolve(cv, v);
#pragma unroll
      for (int r = 0; r < RB; ++r) {
        if (first + r >= end) break;
        T* dst = dest(first + r);
        if (pair) {
          const float2 cs = a.rope[(long long)(start + first + r - r0) * np + i];
          dst[cu] = from_f<T>((u[r] * cs.x - v[r] * cs.y) * tf);
          dst[cv] = from_f<T>((v[r] * cs.x + u[r] * cs.y) * tf);
        } else {
          dst[cu] = from_f<T>(u[r] * tf);
        }
      }
    }
    for (int j = w + lane; j < a.P; j += 32)
      for (int r = first; r < end; ++r) dest(r)[j] = from_f<T>(0.f);
    row = end;
  }
}

// The same for many rows: a thread takes four channels of `rep` times RB rows, with the four they are rotated with.
// Filters of at most four taps; d, vd, rd / 2 and the source's pitch multiples of 4.  grid (ceil(items / 256),
// ceil(M / (rep RB))): items of a row are the rotated quads of all heads, the unrotated ones, the values'
template <typename T, int RB>
__global__ void __launch_bounds__(256) attn_inputs4_kernel(ConvIn<T, Mat<T>, false> in, PagedAttnArgs a, int qk_heads, int items, int rep) {
  const int it = blockIdx.x * 256 + threadIdx.x;
  if (it >= items) return;
  const int np = a.rd / 2, nr = np / 4, nu = (a.d - a.rd) / 4, nv = a.vd / 4;
  int head, c;                                             // head of q | k | v; first channel in it
  const bool pair = it < qk_heads * nr;
  bool is_v = false;
  if (pair) { head = it / nr; c = it % nr * 4; }
  else if (it < qk_heads * (nr + nu)) { const int i = it - qk_heads * nr; head = i / nu; c = a.rd + i % nu * 4; }
  else { const int i = it - qk_heads * (nr + nu); is_v = true; head = i / nv; c = i % nv * 4; }
  const int col = is_v ? (a.H + a.KH) * a.d + head * a.vd + c : head * a.d + c;
  const float tf = !is_v && head < a.H && a.temp ? a.temp[head] : 1.f;
  int row = blockIdx.y * rep * RB;
  const int last = min(row + rep * RB, a.rows.M);
  float wu[4][4], wv[4][4];
  in.filters4(col, wu);
  in.filters4(pair ? col + np : col, wv);
#pragma unroll 1
  while (row < last) {                                     // stretches of one entry
    int slot, r0, n, start;
    a.rows.entry(a.rows.entry_of(row), &slot, &r0, &n, &start);
    const int end = min(min(last, row + RB), r0 + n);
    float4 u[RB], v[RB];
    in.template run4<RB>(row, end, r0, start, slot, col, wu, u);
    if (pair) in.template run4<RB>(row, end, r0, start, slot, col + np, wv, v);
#pragma unroll
    for (int r = 0; r < RB; ++r) {
      if (row + r >= end) break;
      const int pos = start + row + r - r0;
      T* dst;
      if (!is_v && head < a.H) {
        dst = reinterpret_cast<T*>(a.q) + ((long long)(row + r) * a.H + head) * a.P + c;
      } else {
        const int g = is_v ? head : head - a.H;
        dst = reinterpret_cast<T*>(is_v ? a.vplane : a.kplane) +
              (((long long)a.table[(long long)slot * a.max_pages + pos / KV_PAGE] * KV_PAGE + pos % KV_PAGE) * a.KH + g) * a.P + c;
      }
      if (pair) {
        const float4* cs = reinterpret_cast<const float4*>(a.rope + (long long)pos * np + c);   // two pairs each
        const float4 p0 = cs[0], p1 = cs[1], x = scaled(u[r], tf), y = scaled(v[r], tf);
        store4(dst, make_float4(x.x * p0.x - y.x * p0.y, x.y * p0.z - y.y * p0.w, x.z * p1.x - y.z * p1.y, x.w * p1.z - y.w * p1.w));
        store4(dst + np, make_float4(y.x * p0.x + x.x * p0.y, y.y * p0.z + x.y * p0.w, y.z * p1.x + x.z * p1.y, y.w * p1.z + x.w * p1.w));
      } else {
        store4(dst, scaled(u[r], tf));
      }
      const int w = is_v ? a.vd : a.d;
      if (c + 4 == w || (pair && np + c + 4 == w))         // the last quad of a head also pads it
        for (int j = w - (pair ? np + c : c); j < a.P - (pair ? np + c : c); j += 4) store4((pair ? dst + np : dst) + j, make_float4(0.f, 0.f, 0.f, 0.f));
      if (n <= a.pending && in.taps > 1)
        for (int e = 0; e < 4; ++e) {
          in.keep(slot, pos, col + e, in.src.get(row + r, in.col0 + col + e));
          if (pair) in.keep(slot, pos, col + np + e, in.src.get(row + r, in.col0 + col + np + e));
        }
    }
    row = end;
  }
}

// The same without convolutions: a thread takes four channels of one row (with the four they are rotated with) in up to `per`
// heads, four at a time.  d, vd, rd / 2 and the source's pitch multiples of 4; bias [channels] or null.
// grid (ceil(M max(quads of a head) / 256), slices of the query and key heads, and one of the values)
template <typename T, typename S>
__global__ void __launch_bounds__(256) attn_rows4_kernel(S src, const float* __restrict__ bias, PagedAttnArgs a, int qk_heads, int per) {
  const int np = a.rd / 2, nr = np / 4;
  const bool is_v = a.own_kv && blockIdx.y == gridDim.y - 1;
  const int w = is_v ? a.vd : a.d, quads = is_v ? a.vd / 4 : nr + (a.d - a.rd) / 4;
  const long long t = (long long)blockIdx.x * 256 + threadIdx.x;
  const int row = (int)(t / quads), i = (int)(t % quads);
  if (row >= a.rows.M) return;
  const bool pair = !is_v && i < nr;
  const int c = is_v || pair ? 4 * i : a.rd + 4 * (i - nr), col0 = is_v ? (a.H + a.KH) * a.d : 0;
  const int last = is_v ? a.KH : min(qk_heads, ((int)blockIdx.y + 1) * per);
  int slot, r0, n, start;
  a.rows.entry(a.rows.entry_of(row), &slot, &r0, &n, &start);
  const int pos = start + row - r0;
  const long long page = ((long long)a.table[(long long)slot * a.max_pages + pos / KV_PAGE] * KV_PAGE + pos % KV_PAGE) * a.KH;
  float4 p0 = make_float4(1.f, 0.f, 1.f, 0.f), p1 = p0;
  if (pair) {
    const float4* cs = reinterpret_cast<const float4*>(a.rope + (long long)pos * np + c);          // two pairs each
    p0 = cs[0]; p1 = cs[1];
  }
  const bool pads = a.P > w && (c + 4 == w || (pair && np + c + 4 == w));       // the last quad of a head also pads it
#pragma unroll 1
  for (int head = is_v ? 0 : blockIdx.y * per; head < last; head += 4) {
    float4 x[4], y[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int col = col0 + min(head + k, last - 1) * w + c;
      x[k] = get4(src, row, col);
      if (pair) y[k] = get4(src, row, col + np);
    }
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int h = head + k;
      if (h >= last) break;
      const int col = col0 + h * w + c;
      const bool is_q = !is_v && h < a.H;
      const float tf = is_q && a.temp ? a.temp[h] : 1.f;
      T* dst = is_q ? reinterpret_cast<T*>(a.q) + ((long long)row * a.H + h) * a.P + c
                    : reinterpret_cast<T*>(is_v ? a.vplane : a.kplane) + (page + (is_v ? h : h - a.H)) * a.P + c;
      auto value = [&](float4 v, int at) {
        v = make_float4(round_to<T>(v.x), round_to<T>(v.y), round_to<T>(v.z), round_to<T>(v.w));
        if (bias) { const float4 b = load4(bias + at); v = make_float4(v.x + b.x, v.y + b.y, v.z + b.z, v.w + b.w); }
        return scaled(v, tf);
      };
      const float4 u = value(x[k], col);
      if (pair) {
        const float4 v = value(y[k], col + np);
        store4(dst, make_float4(u.x * p0.x - v.x * p0.y, u.y * p0.z - v.y * p0.w, u.z * p1.x - v.z * p1.y, u.w * p1.z - v.w * p1.w));
        store4(dst + np, make_float4(v.x * p0.x + u.x * p0.y, v.y * p0.z + u.y * p0.w, v.z * p1.x + u.z * p1.y, v.w * p1.z + u.w * p1.w));
      } else {
        store4(dst, u);
      }
      if (pads)
        for (int j = w - c; j < a.P - c; j += 4) store4(dst + j, make_float4(0.f, 0.f, 0.f, 0.f));
    }
  }
}

// Heads with a norm (or with interleaved pairs and biases), without convolutions: bias, norm, rotation.  One warp per (row, unit) with the
// head staged in shared memory; units as above.  grid (units, ceil(M / 8)), block (32, 8), 8 max(d, vd) floats
template <typename T, typename S>
__global__ void __launch_bounds__(256) attn_heads_kernel(ConvIn<T, S, false> in, PagedAttnArgs a) {
  extern __shared__ __align__(16) float s_head[];
  const int lane = threadIdx.x, unit = blockIdx.x, row = blockIdx.y * 8 + threadIdx.y;
  if (row >= a.rows.M) return;
  float* s = s_head + threadIdx.y * max(a.d, a.vd);
  const bool is_q = unit < a.H, is_v = unit >= a.H + a.KH;
  const int head = is_q ? unit : is_v ? unit - a.H - a.KH : unit - a.H, w = is_v ? a.vd : a.d, np = is_v ? 0 : a.rd / 2;
  const int c0 = is_v ? (a.H + a.KH) * a.d + head * a.vd : unit * a.d;
  const float* nw = is_v ? nullptr : is_q ? a.qn : a.kn;
  int slot, r0, n, start;
  a.rows.entry(a.rows.entry_of(row), &slot, &r0, &n, &start);
  const int pos = start + row - r0;
  float ss = 0.f;
  for (int c = lane; c < w; c += 32) {
    const float v = round_to<T>(in.src.get(row, in.col0 + c0 + c)) + (in.bias ? in.bias[c0 + c] : 0.f);
    s[c] = v;
    ss += v * v;
  }
  const float r = nw ? 1.f / sqrtf(warp_sum(ss) / (float)w + a.eps) : 1.f;
  __syncwarp();
  T* dst = is_q ? reinterpret_cast<T*>(a.q) + ((long long)row * a.H + head) * a.P
                : reinterpret_cast<T*>(is_v ? a.vplane : a.kplane) +
                      (((long long)a.table[(long long)slot * a.max_pages + pos / KV_PAGE] * KV_PAGE + pos % KV_PAGE) * a.KH + head) * a.P;
  const float tf = is_q && a.temp ? a.temp[head] : 1.f;
  auto value = [&](int c) { return nw ? s[c] * r * nw[c] * tf : s[c] * tf; };
  for (int i = lane; i < w - np; i += 32) {
    if (i < np) {
      const int cu = a.interleaved ? 2 * i : i, cv = a.interleaved ? 2 * i + 1 : np + i;
      const float u = value(cu), v = value(cv);
      const float2 cs = a.rope[(long long)pos * np + i];
      dst[cu] = from_f<T>(u * cs.x - v * cs.y);
      dst[cv] = from_f<T>(v * cs.x + u * cs.y);
    } else {
      dst[np + i] = from_f<T>(value(np + i));
    }
  }
  for (int c = w + lane; c < a.P; c += 32) dst[c] = from_f<T>(0.f);
}

// The same for interleaved pairs and heads of at most 128: W lanes take a head, four channels each, of RB rows at once.
// d, vd, rd and the source's pitch multiples of 4.  grid (ceil(units / (32 / W)), ceil(M / (8 RB))), block (32, 8)
template <typename T, typename S, int W, int RB>
__global__ void __launch_bounds__(256) attn_heads4_kernel(ConvIn<T, S, false> in, PagedAttnArgs a, int units) {
  const int l = threadIdx.x % W, unit = blockIdx.x * (32 / W) + threadIdx.x / W, row0 = (blockIdx.y * 8 + threadIdx.y) * RB;
  if (row0 >= a.rows.M) return;
  const bool live = unit < units, is_q = unit < a.H, is_v = unit >= a.H + a.KH;
  const int head = is_q ? unit : is_v ? unit - a.H - a.KH : unit - a.H, w = is_v ? a.vd : a.d, np = is_v ? 0 : a.rd / 2, c = 4 * l;
  const int c0 = (is_v ? (a.H + a.KH) * a.d + head * a.vd : unit * a.d) + c;
  const float* nw = is_v ? nullptr : is_q ? a.qn : a.kn;
  const bool mine = live && c < w;
  float4 x[RB], b = make_float4(0.f, 0.f, 0.f, 0.f), wt = make_float4(1.f, 1.f, 1.f, 1.f);
#pragma unroll
  for (int r = 0; r < RB; ++r)
    x[r] = mine ? get4(in.src, min(row0 + r, a.rows.M - 1), in.col0 + c0) : make_float4(0.f, 0.f, 0.f, 0.f);
  if (mine && in.bias) b = load4(in.bias + c0);
  if (mine && nw) wt = load4(nw + c);
  const float tf = live && is_q && a.temp ? a.temp[head] : 1.f;
  float ss[RB];
#pragma unroll
  for (int r = 0; r < RB; ++r) {
    x[r] = make_float4(round_to<T>(x[r].x) + b.x, round_to<T>(x[r].y) + b.y, round_to<T>(x[r].z) + b.z, round_to<T>(x[r].w) + b.w);
    ss[r] = x[r].x * x[r].x + x[r].y * x[r].y + x[r].z * x[r].z + x[r].w * x[r].w;
  }
#pragma unroll
  for (int o = W / 2; o > 0; o >>= 1)
#pragma unroll
    for (int r = 0; r < RB; ++r) ss[r] += __shfl_xor_sync(0xffffffffu, ss[r], o);
#pragma unroll
  for (int r = 0; r < RB; ++r) {
    const int row = row0 + r;
    if (row >= a.rows.M || !live || c >= a.P) break;
    int slot, r0, n, start;
    a.rows.entry(a.rows.entry_of(row), &slot, &r0, &n, &start);
    const int pos = start + row - r0;
    T* dst = is_q ? reinterpret_cast<T*>(a.q) + ((long long)row * a.H + head) * a.P
                  : reinterpret_cast<T*>(is_v ? a.vplane : a.kplane) +
                        (((long long)a.table[(long long)slot * a.max_pages + pos / KV_PAGE] * KV_PAGE + pos % KV_PAGE) * a.KH + head) * a.P;
    float4 v = x[r];
    if (nw) {
      const float f = 1.f / sqrtf(ss[r] / (float)w + a.eps);
      v = make_float4(v.x * f * wt.x, v.y * f * wt.y, v.z * f * wt.z, v.w * f * wt.w);
    }
    if (c < 2 * np) {
      const float4 cs = *reinterpret_cast<const float4*>(a.rope + (long long)pos * np + 2 * l);
      v = make_float4(v.x * cs.x - v.y * cs.y, v.y * cs.x + v.x * cs.y, v.z * cs.z - v.w * cs.w, v.w * cs.z + v.z * cs.w);
    }
    store4(dst + c, scaled(v, tf));                        // pads too: their quads are zero
  }
}

// ---- one warp per (row, head), any dtype; NR = values per lane (P <= 32 NR).  grid (M, ceil(H / 8)) --------------------
template <typename T, typename S, int NR>
__global__ void __launch_bounds__(256) paged_attn_kernel(PagedAttnArgs a, S proj) {
  const int h = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, row = blockIdx.x;
  if (h >= a.H) return;
  int slot, r0, n, start;
  a.rows.entry(a.rows.entry_of(row), &slot, &r0, &n, &start);
  const int pos = start + row - r0, g = h / (a.H / a.KH);
  const int lo = a.first_key(pos);
  const T* q = reinterpret_cast<const T*>(a.q) + ((long long)row * a.H + h) * a.P;
  const int* tab = a.table + (long long)slot * a.max_pages;
  float qv[NR], acc[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int j = lane + 32 * i;
    qv[i] = j < a.d ? to_f<T>(q[j]) : 0.f;
    acc[i] = 0.f;
  }
  float m = -CUDART_INF_F, l = 0.f;
#pragma unroll 1
  for (int p = lo; p <= pos; ++p) {
    const long long at = (((long long)tab[p / KV_PAGE] * KV_PAGE + p % KV_PAGE) * a.KH + g) * a.P;
    const T *k = reinterpret_cast<const T*>(a.kplane) + at, *v = reinterpret_cast<const T*>(a.vplane) + at;
    float vv[NR], s = 0.f;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int j = lane + 32 * i;
      s = fmaf(qv[i], j < a.d ? to_f<T>(k[j]) : 0.f, s);
      vv[i] = j < a.vd ? to_f<T>(v[j]) : 0.f;
    }
    s = warp_sum(s) * a.scale;
    if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
    const float m2 = fmaxf(m, s), f = expf(m - m2), e = expf(s - m2);
    l = l * f + e;
#pragma unroll
    for (int i = 0; i < NR; ++i) acc[i] = fmaf(acc[i], f, e * vv[i]);
    m = m2;
  }
  T* o = reinterpret_cast<T*>(a.out) + ((long long)row * a.H + h) * a.vd;
  const bool each = a.col_g >= 0 && !a.gate_head;
  if (a.gate_head) l /= sigmoid_f(proj.get_rare(row, a.col_g + h));
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int j = lane + 32 * i;
    if (j < a.vd) o[j] = from_f<T>(acc[i] / l * (each ? sigmoid_f(proj.get_rare(row, a.col_g + h * a.vd + j)) : 1.f));
  }
}

// ---- tensor-core kernel (bf16) ---------------------------------------------------------------------------------------
// A CTA of W warps takes 16 W rows of one key/value head of one entry (row f = token * group + head of the group) and walks
// the key pages those tokens see, double-buffered through cp.async; every warp keeps 16 rows' soft-max and output.
template <int P, int W>
__host__ __device__ constexpr int mma_smem() {
  return (4 * KV_PAGE + (P > 128 ? 16 * W : 0)) * (P + 8) * 2;
}

template <int P, int W, typename S>
__global__ void __launch_bounds__(32 * W) paged_attn_mma_kernel(PagedAttnArgs a, S proj) {
  using namespace mma_detail;
  constexpr int LD = P + 8, ROWS = 16 * W, TH = 32 * W, CH = P / 8;
  constexpr bool QREG = P <= 128;                        // query fragments in registers, or read from shared memory each page
  static_assert(!QREG || ROWS <= 2 * KV_PAGE, "the query tile is staged where the values go");
  static_assert(ROWS * P * 4 <= 4 * KV_PAGE * LD * 2, "the output tile is staged where keys and values were");
  extern __shared__ __align__(16) unsigned char raw[];
  bf16* sK = reinterpret_cast<bf16*>(raw);               // [2][KV_PAGE][LD]
  bf16* sV = sK + 2 * KV_PAGE * LD;
  bf16* sQ = QREG ? sV : sV + 2 * KV_PAGE * LD;
  int slot, r0, n, start;
  a.rows.entry(blockIdx.z, &slot, &r0, &n, &start);
  const int hg = a.H / a.KH, g = blockIdx.y, f0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * ROWS, nf = n * hg;
  if (f0 >= nf) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int f_last = min(f0 + ROWS, nf) - 1;
  const int p_lo = start + f0 / hg, p_hi = start + f_last / hg;
  const int pg0 = a.first_key(p_lo) / KV_PAGE, pg1 = p_hi / KV_PAGE + 1;
  const int* tab = a.table + (long long)slot * a.max_pages;
  const long long ldp = (long long)a.KH * P;
  const bf16 *kp = reinterpret_cast<const bf16*>(a.kplane) + (long long)g * P, *vp = reinterpret_cast<const bf16*>(a.vplane) + (long long)g * P;
  for (int i = tid; i < ROWS * CH; i += TH) {
    const int r = i / CH, c = (i % CH) * 8, f = f0 + r;
    const bool ok = f < nf;
    const bf16* q = reinterpret_cast<const bf16*>(a.q) + ((long long)(r0 + (ok ? f / hg : 0)) * a.H + g * hg + (ok ? f % hg : 0)) * P + c;
    cp_async16(sQ + r * LD + c, q, ok);
  }
  cp_async_commit();
  auto fetch = [&](int pg, int buf) {
    const long long base = (long long)tab[pg] * KV_PAGE * ldp;
    const int valid = min(KV_PAGE, p_hi + 1 - pg * KV_PAGE);       // keys beyond the tile's last position: zero
    for (int i = tid; i < KV_PAGE * CH; i += TH) {
      const int r = i / CH, c = (i % CH) * 8;
      const bool ok = r < valid;
      const long long at = base + (ok ? r : 0) * ldp + c;
      cp_async16(sK + (buf * KV_PAGE + r) * LD + c, kp + at, ok);
      cp_async16(sV + (buf * KV_PAGE + r) * LD + c, vp + at, ok);
    }
    cp_async_commit();
  };
  unsigned qf[QREG ? P / 16 : 1][4];
  const bf16* q_at = sQ + (16 * warp + (lane & 15)) * LD + ((lane >> 4) << 3);
  if (QREG) {
    cp_async_wait<0>();
    __syncthreads();
#pragma unroll
    for (int k = 0; k < (QREG ? P / 16 : 1); ++k) ldmatrix_x4(qf[k][0], qf[k][1], qf[k][2], qf[k][3], q_at + 16 * k);
    __syncthreads();
  }
  float acc[P / 8][4];
#pragma unroll
  for (int j = 0; j < P / 8; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
  float m_run[2] = {-CUDART_INF_F, -CUDART_INF_F}, l_run[2] = {0.f, 0.f};
  int rp[2], rk[2];                                       // positions of rows lane / 4 and lane / 4 + 8 (-1 beyond the entry), their first keys
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int f = f0 + 16 * warp + (lane >> 2) + 8 * e;
    rp[e] = f < nf ? start + f / hg : -1;
    rk[e] = f < nf ? a.first_key(rp[e]) : 0;
  }
  const int w_lo = start + min(f0 + 16 * warp, nf - 1) / hg, w_hi = start + min(f0 + 16 * warp + 15, nf - 1) / hg;
  const int k_lo = a.first_key(w_lo), k_hi = a.first_key(w_hi);
  const float sc = a.softcap > 0.f ? 1.f : a.scale * 1.4426950408889634f;
  fetch(pg0, 0);
  for (int pg = pg0, buf = 0; pg < pg1; ++pg, buf ^= 1) {
    if (pg + 1 < pg1) { fetch(pg + 1, buf ^ 1); cp_async_wait<1>(); } else cp_async_wait<0>();
    __syncthreads();
    const bf16 *K = sK + buf * KV_PAGE * LD, *V = sV + buf * KV_PAGE * LD;
    // nothing of this page is visible to the warp's rows: keys all later, or all before the first one
    const bool skip = pg * KV_PAGE > w_hi || pg * KV_PAGE + KV_PAGE <= k_lo;
    if (!skip) {
      float s[8][4];
#pragma unroll
      for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[j][e] = 0.f;
#pragma unroll
      for (int k = 0; k < P / 16; ++k) {
        unsigned af[4];
        if (QREG) {
#pragma unroll
          for (int e = 0; e < 4; ++e) af[e] = qf[QREG ? k : 0][e];
        } else {
          ldmatrix_x4(af[0], af[1], af[2], af[3], q_at + 16 * k);
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          unsigned b0[2], b1[2];
          const int r = 16 * j + (lane & 7) + ((lane >> 4) << 3), c = 16 * k + (((lane >> 3) & 1) << 3);
          ldmatrix_x4(b0[0], b0[1], b1[0], b1[1], K + r * LD + c);
          mma_bf16(s[2 * j], af, b0);
          mma_bf16(s[2 * j + 1], af, b1);
        }
      }
      const bool whole = pg * KV_PAGE + KV_PAGE - 1 <= w_lo && pg * KV_PAGE >= k_hi;
      float mx[2] = {m_run[0], m_run[1]};
      if (a.softcap > 0.f)
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
          for (int x = 0; x < 4; ++x) s[j][x] = softcap_log2(s[j][x] * a.scale, a.softcap);
#pragma unroll
      for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const int e = x >> 1;
          float v = s[j][x] * sc;
          if (!whole) {
            const int key = pg * KV_PAGE + 8 * j + (lane & 3) * 2 + (x & 1);
            if (key > rp[e] || key < rk[e]) v = -CUDART_INF_F;
          }
          s[j][x] = v;
          mx[e] = fmaxf(mx[e], v);
        }
      float f[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 1));
        mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 2));
        f[e] = mx[e] == -CUDART_INF_F ? 1.f : exp2f(m_run[e] - mx[e]);
        m_run[e] = mx[e];
        if (mx[e] == -CUDART_INF_F) mx[e] = 0.f;          // nothing seen yet: every weight becomes exp2(-inf) = 0
        l_run[e] *= f[e];
      }
#pragma unroll
      for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          s[j][x] = exp2f(s[j][x] - mx[x >> 1]);
          l_run[x >> 1] += s[j][x];                       // this lane's share; the four lanes of a row are summed at the end
        }
#pragma unroll
      for (int j = 0; j < P / 8; ++j) { acc[j][0] *= f[0]; acc[j][1] *= f[0]; acc[j][2] *= f[1]; acc[j][3] *= f[1]; }
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const unsigned af[4] = {pack_bf16(s[2 * k][0], s[2 * k][1]), pack_bf16(s[2 * k][2], s[2 * k][3]),
                                pack_bf16(s[2 * k + 1][0], s[2 * k + 1][1]), pack_bf16(s[2 * k + 1][2], s[2 * k + 1][3])};
#pragma unroll
        for (int j = 0; j < P / 16; ++j) {
          unsigned b0[2], b1[2];
          const int r = 16 * k + (lane & 7) + (((lane >> 3) & 1) << 3), c = 16 * j + ((lane >> 4) << 3);
          ldmatrix_x4_t(b0[0], b0[1], b1[0], b1[1], V + r * LD + c);
          mma_bf16(acc[2 * j], af, b0);
          mma_bf16(acc[2 * j + 1], af, b1);
        }
      }
    }
    __syncthreads();
  }
  // through shared memory, so that rows are gated and stored in whole lines
  float* sO = reinterpret_cast<float*>(raw) + 16 * warp * P;
  const int fw = f0 + 16 * warp;
  const bool each = a.col_g >= 0 && !a.gate_head;         // a gate per element, else per head or none
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    float l = l_run[e];
    l += __shfl_xor_sync(0xffffffffu, l, 1);
    l += __shfl_xor_sync(0xffffffffu, l, 2);
    float inv = 1.f / l;
    const int f = fw + (lane >> 2) + 8 * e;
    if (a.gate_head && f < nf) inv *= sigmoid_f(proj.get_rare(r0 + f / hg, a.col_g + g * hg + f % hg));
#pragma unroll
    for (int j = 0; j < P / 8; ++j)
      *reinterpret_cast<float2*>(sO + ((lane >> 2) + 8 * e) * P + 8 * j + (lane & 3) * 2) = make_float2(acc[j][2 * e] * inv, acc[j][2 * e + 1] * inv);
  }
  __syncwarp();
  if (a.vd % 4 == 0 && (!each || (a.col_g % 4 == 0 && proj.ld % 4 == 0))) {
    // four columns per lane, eight rows' gates requested at a time
#pragma unroll 1
    for (int c = lane * 4; c < a.vd; c += 128)
#pragma unroll 1
      for (int r = 0; r < 16; r += 8) {
        float4 gt[8];
#pragma unroll
        for (int y = 0; y < 8; ++y) {
          const int f = min(fw + r + y, nf - 1);
          if (each) gt[y] = get4(proj, r0 + f / hg, a.col_g + (g * hg + f % hg) * a.vd + c);
        }
#pragma unroll
        for (int y = 0; y < 8; ++y) {
          const int f = fw + r + y;
          if (f >= nf) break;
          float4 v = load4(sO + (r + y) * P + c);
          if (each) { v.x *= sigmoid_f(gt[y].x); v.y *= sigmoid_f(gt[y].y); v.z *= sigmoid_f(gt[y].z); v.w *= sigmoid_f(gt[y].w); }
          store4(reinterpret_cast<bf16*>(a.out) + ((long long)(r0 + f / hg) * a.H + g * hg + f % hg) * a.vd + c, v);
        }
      }
    return;
  }
  for (int r = 0; r < 16; ++r) {
    const int f = fw + r;
    if (f >= nf) break;
    const long long row = r0 + f / hg;
    const int h = g * hg + f % hg;
    bf16* o = reinterpret_cast<bf16*>(a.out) + (row * a.H + h) * a.vd;
    for (int c = lane; c < a.vd; c += 32)
      o[c] = __float2bfloat16_rn(sO[r * P + c] * (each ? sigmoid_f(proj.get_rare(row, a.col_g + h * a.vd + c)) : 1.f));
  }
}

template <int P, int W, typename S>
int32_t launch_mma(vn_ctx* ctx, const PagedAttnArgs& a, const S& proj) {
  static unsigned long long done = 0;
  if (!((done >> (ctx->device & 63)) & 1ull)) {
    VN_CUDA(ctx, cudaFuncSetAttribute((paged_attn_mma_kernel<P, W, S>), cudaFuncAttributeMaxDynamicSharedMemorySize, (mma_smem<P, W>())));
    done |= 1ull << (ctx->device & 63);
  }
  const dim3 grid(ceil_div(a.rows.max_n * (a.H / a.KH), 16 * W), a.KH, a.rows.n_ent);
  VN_LAUNCH_NAMED(ctx, "paged_attn_mma_kernel", (paged_attn_mma_kernel<P, W, S>), grid, 32 * W, (mma_smem<P, W>()), a, proj);
  return VN_OK;
}

template <typename T, typename S>
int32_t launch_simt(vn_ctx* ctx, const PagedAttnArgs& a, const S& proj) {
  const dim3 grid(a.rows.M, ceil_div(a.H, 8));
  const int nr = a.P / 32;
#define PA(NR) VN_LAUNCH_NAMED(ctx, "paged_attn_kernel", (paged_attn_kernel<T, S, NR>), grid, 256, 0, a, proj)
  if (nr <= 2) PA(2); else if (nr <= 4) PA(4); else if (nr <= 8) PA(8); else PA(32);
#undef PA
  return VN_OK;
}

template <typename S>
int32_t pick_mma(vn_ctx* ctx, const PagedAttnArgs& a, const S& proj) {
  // eight warps share a page where there are tiles enough for it
  const bool wide = (long long)ceil_div(a.rows.max_n * (a.H / a.KH), 128) * a.KH * a.rows.n_ent >= 2 * ctx->sm_count;
#define MM(P) return wide ? launch_mma<P, 8>(ctx, a, proj) : launch_mma<P, 4>(ctx, a, proj)
  switch (a.P) {
    case 32: MM(32);
    case 64: MM(64);
    case 96: MM(96);
    case 128: MM(128);
    case 192: return launch_mma<192, 4>(ctx, a, proj);
    case 256: return launch_mma<256, 4>(ctx, a, proj);
    default: return vn_fail(ctx, VN_ERR_UNSUPPORTED, "key pitch %d", a.P);
  }
#undef MM
}

}  // namespace

int32_t vn_rope_table(vn_ctx* ctx, const double* freq_dev, int pairs, float amp, int rows, float2* out) {
  const long long total = (long long)pairs * rows;
  if (total <= 0) return VN_OK;
  VN_LAUNCH(ctx, rope_table_kernel, (unsigned)ceil_div(total, 128ll), 128, 0, freq_dev, pairs, amp, total, out);
  return VN_OK;
}

template <typename T, typename S>
int32_t vn_attn_inputs(vn_ctx* ctx, const ConvIn<T, S, false>& conv, const PagedAttnArgs& a) {
  const int units = a.H + (a.own_kv ? 2 * a.KH : 0);
  const dim3 block(32, 8);
  if (a.qn || (conv.bias && a.interleaved)) {
    VN_REQUIRE(ctx, conv.taps == 1, "norms and biases of the heads stand without convolutions");
    const int w = std::max(a.d, a.vd);
    if (a.d % 4 == 0 && a.vd % 4 == 0 && a.rd % 4 == 0 && conv.src.ld % 4 == 0 && w <= 128 && (a.interleaved || !a.rd)) {
      const bool many = a.rows.M >= 512;
#define HEADS(W, RB) VN_LAUNCH_NAMED(ctx, "attn_heads_kernel", (attn_heads4_kernel<T, S, W, RB>), \
                                     dim3(ceil_div(units, 32 / W), ceil_div(a.rows.M, 8 * RB)), block, 0, conv, a, units)
#define HEADS1(W) do { if (many) HEADS(W, 4); else HEADS(W, 1); } while (0)
      if (w <= 32) HEADS1(8); else if (w <= 64) HEADS1(16); else HEADS1(32);
#undef HEADS1
#undef HEADS
      return VN_OK;
    }
    VN_LAUNCH_NAMED(ctx, "attn_heads_kernel", (attn_heads_kernel<T, S>), dim3(units, ceil_div(a.rows.M, 8)), block, (size_t)8 * w * 4, conv, a);
    return VN_OK;
  }
  if (!conv.named && conv.taps == 1 && a.d % 4 == 0 && a.vd % 4 == 0 && a.rd % 8 == 0 && conv.src.ld % 4 == 0 && !a.interleaved) {
    const int qk = a.H + (a.own_kv ? a.KH : 0), quads = std::max((a.d - a.rd / 2) / 4, a.own_kv ? a.vd / 4 : 0);
    const long long blocks = ceil_div((long long)a.rows.M * quads, 256ll);
    int per = 4;                                           // more heads per thread where there are threads enough
    while (per < qk && blocks * ceil_div(qk, 2 * per) >= 8ll * ctx->sm_count) per *= 2;
    VN_LAUNCH_NAMED(ctx, "attn_inputs_kernel", (attn_rows4_kernel<T, S>), dim3((unsigned)blocks, ceil_div(qk, per) + (a.own_kv ? 1 : 0)), 256, 0, conv.src, conv.bias, a, qk, per);
    return VN_OK;
  }
  if constexpr (std::is_same<S, Mat<T>>::value) {
    if (conv.taps <= 4 && a.d % 4 == 0 && a.vd % 4 == 0 && a.rd % 8 == 0 && conv.src.ld % 4 == 0 && !a.interleaved) {
      const int rep = a.rows.M >= 2048 ? 4 : 1;
      const int qk = a.H + (a.own_kv ? a.KH : 0), items = qk * (a.d - a.rd / 2) / 4 + (a.own_kv ? a.KH * a.vd / 4 : 0);
      VN_LAUNCH_NAMED(ctx, "attn_inputs_kernel", (attn_inputs4_kernel<T, 4>), dim3(ceil_div(items, 256), ceil_div(a.rows.M, 4 * rep)), 256, 0, conv, a, qk, items, rep);
      return VN_OK;
    }
  }
  if (a.rows.M >= 512 && conv.taps <= 4)
    VN_LAUNCH_NAMED(ctx, "attn_inputs_kernel", (attn_inputs_kernel<T, S, 8>), dim3(units, ceil_div(a.rows.M, 64)), block, 0, conv, a);
  else
    VN_LAUNCH_NAMED(ctx, "attn_inputs_kernel", (attn_inputs_kernel<T, S, 1>), dim3(units, ceil_div(a.rows.M, 8)), block, 0, conv, a);
  return VN_OK;
}
template int32_t vn_attn_inputs(vn_ctx*, const ConvIn<float, Src, false>&, const PagedAttnArgs&);
template int32_t vn_attn_inputs(vn_ctx*, const ConvIn<bf16, Src, false>&, const PagedAttnArgs&);
template int32_t vn_attn_inputs(vn_ctx*, const ConvIn<bf16, Mat<bf16>, false>&, const PagedAttnArgs&);

template <> int32_t vn_paged_attention<float, Src>(vn_ctx* ctx, const Src& proj, const PagedAttnArgs& a, bool) {
  return launch_simt<float>(ctx, a, proj);
}
template <> int32_t vn_paged_attention<bf16, Src>(vn_ctx* ctx, const Src& proj, const PagedAttnArgs& a, bool mma) {
  return mma ? pick_mma(ctx, a, proj) : launch_simt<bf16>(ctx, a, proj);
}
template <> int32_t vn_paged_attention<bf16, Mat<bf16>>(vn_ctx* ctx, const Mat<bf16>& proj, const PagedAttnArgs& a, bool mma) {
  return mma ? pick_mma(ctx, a, proj) : launch_simt<bf16>(ctx, a, proj);
}
