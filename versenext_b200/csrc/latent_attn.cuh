// Latent attention: one cached vector c of kv_rank values per token serves as key and value of every head.
//
// With k_h = W_uk,h c and v_h = W_uv,h c the score (q_h . k_h) equals (W_uk,h^T q_h) . c and the output W_uv,h (sum_j p_j
// c_j), so the queries are carried into the latent space once and attention runs on c itself (all heads share the keys:
// heads and tokens together are the rows of one matrix product).  Sliding window, a learned sink per head in the
// denominator, an output gate per head; scores, soft-max and gate in fp32.  A key may have a rotated part that all heads
// share: it stands behind the latent in the cached row, the query's rotated part behind the carried query.
//
// Cache: pages of KV_PAGE tokens, plane[page * KV_PAGE + pos % KV_PAGE][Rp]; table[slot * max_pages + pos / KV_PAGE].
#pragma once
#include "gemm_mma.cuh"
#include "rows.cuh"
#include <math_constants.h>

struct LatentArgs {
  const void* qc = nullptr;       // [M, H, Rp] queries in the latent space, storage dtype
  const void* plane = nullptr;    // latent cache of this layer run, storage dtype
  const int* table = nullptr;
  int max_pages = 0, Rp = 0, H = 0;
  int window = 0;                 // position i sees j with 0 <= i - j < window; 0: no limit
  float scale = 1.f;
  const float* sink = nullptr;    // [H] or null
  const float* gate = nullptr;    // [M, H] factors of the heads' outputs, or null
  void* out = nullptr;            // [M, H, Rp] storage dtype
  // key splits (decode): partial results of gridDim.x ranges of key pages, merged by latent_merge_kernel
  int splits = 1;
  float* part_o = nullptr;        // [splits][M * H][Rp] unnormalised
  float* part_ml = nullptr;       // [splits][M * H][2] maximum, sum
  Rows rows;
};

// Inputs of the attention.  src columns: q [H][d | rr] | latent [R] | rotated key [rr] | gates [n_gate]
struct LatentIn {
  int H = 0, d = 0, dp = 0, rr = 0, R = 0, Rp = 0;
  const float2* rope = nullptr;    // [positions][rr / 2]: pairs of neighbours
  const float* norm_w = nullptr;
  float eps = 0.f;
  int n_gate = 0;
  float* gate = nullptr;           // [M, n_gate] sigmoid of the gates, or null
  void* gate_t = nullptr;          // the same in the storage dtype, or null
  void* q = nullptr;               // [M, H, dp] storage dtype
  void* qc = nullptr;              // [M, H, Rp]: columns from R on (rr > 0)
  void* plane = nullptr;
  const int* table = nullptr;
  int max_pages = 0;
};

// latent of the row: RMS norm with a plain weight, appended to its page with the rotated key; queries to the storage dtype
// (head pitch dp), their rotated parts to their places behind the carried queries; sigmoid of the gates.  grid (M, parts): the
// queries and gates are shared out, the first part has the latent
template <typename T, typename S>
__global__ void __launch_bounds__(256) latent_append_kernel(S src, LatentIn a, Rows rows) {
  __shared__ float sm[8];
  const int H = a.H, d = a.d, dp = a.dp, rr = a.rr, R = a.R, Rp = a.Rp, max_pages = a.max_pages, qd = d + rr, np = rr / 2;
  extern __shared__ float s_c[];
  const int row = blockIdx.x;
  int slot, r0, n, start;
  rows.entry(rows.entry_of(row), &slot, &r0, &n, &start);
  const int pos = start + row - r0;
  const int t0 = blockIdx.y * 256 + threadIdx.x, stride = gridDim.y * 256;
  const float2* rope = a.rope + (long long)pos * np;
  // pair i of the rr values from column c on, rotated by the row's position
  auto rotated = [&](int c, int i) {
    const float u = src.get(row, c + 2 * i), v = src.get(row, c + 2 * i + 1);
    const float2 cs = rope[i];
    return make_float2(u * cs.x - v * cs.y, v * cs.x + u * cs.y);
  };
  if (blockIdx.y == 0) {
    float ss = 0.f;
    for (int j = threadIdx.x; j < R; j += 256) {
      const float v = src.get(row, H * qd + j);
      s_c[j] = v;
      ss += v * v;
    }
    const float r = sqrtf(block_sum256(ss, sm) / (float)R + a.eps);
    const int pg = pos / KV_PAGE;
    if (pg < max_pages) {
      T* dst = reinterpret_cast<T*>(a.plane) + ((long long)a.table[(long long)slot * max_pages + pg] * KV_PAGE + pos % KV_PAGE) * Rp;
      for (int j = threadIdx.x; j < Rp; j += 256)
        if (j < R || j >= R + rr) dst[j] = from_f<T>(j < R ? s_c[j] / r * a.norm_w[j] : 0.f);
      for (int i = threadIdx.x; i < np; i += 256) {
        const float2 v = rotated(H * qd + R, i);
        dst[R + 2 * i] = from_f<T>(v.x);
        dst[R + 2 * i + 1] = from_f<T>(v.y);
      }
    }
  }
  T* q = reinterpret_cast<T*>(a.q) + (long long)row * H * dp;
  if (d % 4 == 0 && dp == d && rr % 4 == 0 && R % 4 == 0 && a.n_gate % 4 == 0 && src.ld % 4 == 0) {      // four columns at a time
    for (int i = t0; i < H * d / 4; i += stride) {
      const int h = 4 * i / d, j = 4 * i % d;
      store4(q + 4 * i, get4(src, row, h * qd + j));
    }
    T* qc = reinterpret_cast<T*>(a.qc) + (long long)row * H * Rp + R;
    const int tail = Rp - R;
    if (rr)
      for (int i = t0; i < H * tail / 4; i += stride) {
        const int h = 4 * i / tail, j = 4 * i % tail;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (j < rr) {
          const float4 u = get4(src, row, h * qd + d + j), cs = load4(reinterpret_cast<const float*>(rope + j / 2));
          v = make_float4(u.x * cs.x - u.y * cs.y, u.y * cs.x + u.x * cs.y, u.z * cs.z - u.w * cs.w, u.w * cs.z + u.z * cs.w);
        }
        store4(qc + h * Rp + j, v);
      }
    for (int i = 4 * t0; i < a.n_gate; i += 4 * stride) {
      float4 v = get4(src, row, H * qd + R + rr + i);
      v = make_float4(sigmoid_f(v.x), sigmoid_f(v.y), sigmoid_f(v.z), sigmoid_f(v.w));
      if (a.gate) store4(a.gate + (long long)row * a.n_gate + i, v);
      if (a.gate_t) store4(reinterpret_cast<T*>(a.gate_t) + (long long)row * a.n_gate + i, v);
    }
    return;
  }
  for (int i = t0; i < H * dp; i += stride) {
    const int h = i / dp, j = i % dp;
    q[i] = from_f<T>(j < d ? src.get(row, h * qd + j) : 0.f);
  }
  if (rr) {
    T* qc = reinterpret_cast<T*>(a.qc) + (long long)row * H * Rp;
    for (int i = t0; i < H * np; i += stride) {
      const int h = i / np, j = i % np;
      const float2 v = rotated(h * qd + d, j);
      qc[h * Rp + R + 2 * j] = from_f<T>(v.x);
      qc[h * Rp + R + 2 * j + 1] = from_f<T>(v.y);
    }
    const int pad = Rp - R - rr;
    for (int i = t0; i < H * pad; i += stride) qc[(i / pad) * Rp + R + rr + i % pad] = from_f<T>(0.f);
  }
  for (int i = t0; i < a.n_gate; i += stride) {
    const float v = sigmoid_f(src.get(row, H * qd + R + rr + i));
    if (a.gate) a.gate[(long long)row * a.n_gate + i] = v;
    if (a.gate_t) reinterpret_cast<T*>(a.gate_t)[(long long)row * a.n_gate + i] = from_f<T>(v);
  }
}

// ---- one warp per (row, head), any dtype; NR = values per lane (Rp <= 32 NR).  grid (ceil(H / 8), M) -------------
template <typename T, int NR>
__global__ void __launch_bounds__(256) latent_attn_kernel(LatentArgs a) {
  const int h = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, row = blockIdx.y;
  if (h >= a.H) return;
  int slot, r0, n, start;
  a.rows.entry(a.rows.entry_of(row), &slot, &r0, &n, &start);
  const int pos = start + row - r0;
  const int lo = a.window > 0 ? max(0, pos - a.window + 1) : 0;
  const T* q = reinterpret_cast<const T*>(a.qc) + ((long long)row * a.H + h) * a.Rp;
  const int* tab = a.table + (long long)slot * a.max_pages;
  float qv[NR], acc[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int j = lane + 32 * i;
    qv[i] = j < a.Rp ? to_f<T>(q[j]) : 0.f;
    acc[i] = 0.f;
  }
  float m = a.sink ? a.sink[h] : -CUDART_INF_F, l = a.sink ? 1.f : 0.f;
  for (int p = lo; p <= pos; ++p) {
    const T* c = reinterpret_cast<const T*>(a.plane) + ((long long)tab[p / KV_PAGE] * KV_PAGE + p % KV_PAGE) * a.Rp;
    float cv[NR], s = 0.f;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int j = lane + 32 * i;
      cv[i] = j < a.Rp ? to_f<T>(c[j]) : 0.f;
      s = fmaf(qv[i], cv[i], s);
    }
    s = warp_sum(s) * a.scale;
    const float m2 = fmaxf(m, s), f = expf(m - m2), e = expf(s - m2);
    l = l * f + e;
#pragma unroll
    for (int i = 0; i < NR; ++i) acc[i] = fmaf(acc[i], f, e * cv[i]);
    m = m2;
  }
  const float w = (a.gate ? a.gate[(long long)row * a.H + h] : 1.f) / l;
  T* o = reinterpret_cast<T*>(a.out) + ((long long)row * a.H + h) * a.Rp;
#pragma unroll
  for (int i = 0; i < NR; ++i)
    if (lane + 32 * i < a.Rp) o[lane + 32 * i] = from_f<T>(acc[i] * w);
}

// ---- tensor-core kernel (bf16) -------------------------------------------------------------------------------------
// A CTA of four warps takes 16 MT rows (token-major: row f = token * H + head) of one entry and walks the key pages
// those tokens see.  Per page: warp w scores all rows against keys 16 w .. 16 w + 15 over the whole latent, the warps
// exchange row maxima, the weights go to shared memory in bf16, and warp w accumulates columns [w Rp/4, (w+1) Rp/4) of
// the output: keys and values are the same staged page.  Pages arrive through cp.async, double-buffered.
namespace latent_detail {
__device__ __forceinline__ void ldmatrix_x4_trans(unsigned& r0, unsigned& r1, unsigned& r2, unsigned& r3, const void* p) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(s));
}
constexpr int PLD = KV_PAGE + 8;                                   // row pitch of the weights
__host__ __device__ constexpr int row_tiles(int NT) { return NT > 8 ? 2 : 4; }   // the most row tiles a warp can hold
inline size_t smem_bytes(int MT, int Rp) {
  return (size_t)(16 * MT + 2 * KV_PAGE) * (Rp + 8) * 2 + (size_t)16 * MT * PLD * 2 + (size_t)16 * MT * 4 * 4 * 2;
}
}  // namespace latent_detail

// NT: 8-column tiles of the output per warp (Rp == 32 NT); NT is even or the last odd tile is read with its neighbour
template <int NT, int MT>
__global__ void __launch_bounds__(128) latent_attn_mma_kernel(LatentArgs a) {
  using namespace mma_detail;
  using namespace latent_detail;
  constexpr int Rp = 32 * NT, LD = Rp + 8, ROWS = 16 * MT;
  extern __shared__ __align__(16) unsigned char raw[];
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(raw);
  __nv_bfloat16* sC = sQ + ROWS * LD;                              // [2][KV_PAGE][LD]
  __nv_bfloat16* sP = sC + 2 * KV_PAGE * LD;                       // [ROWS][PLD]
  float* sMax = reinterpret_cast<float*>(sP + ROWS * PLD);         // [4 warps][ROWS]
  float* sSum = sMax + 4 * ROWS;
  int slot, r0, n, start;
  a.rows.entry(blockIdx.z, &slot, &r0, &n, &start);
  const int f0 = blockIdx.y * ROWS, nf = n * a.H;
  if (f0 >= nf) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int f_last = min(f0 + ROWS, nf) - 1;
  const int p_lo = start + f0 / a.H, p_hi = start + f_last / a.H;
  const int k_lo = a.window > 0 ? max(0, p_lo - a.window + 1) : 0;
  int pg0 = k_lo / KV_PAGE, pg1 = p_hi / KV_PAGE + 1;
  if (a.splits > 1) {
    const int per = (pg1 - pg0 + a.splits - 1) / a.splits;
    pg0 += blockIdx.x * per;
    pg1 = min(pg1, pg0 + per);
  }
  const int* tab = a.table + (long long)slot * a.max_pages;
  const __nv_bfloat16* plane = reinterpret_cast<const __nv_bfloat16*>(a.plane);
  constexpr int CH = Rp / 8;                                       // 16-byte chunks of a latent row
  const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(a.qc) + ((long long)r0 * a.H + f0) * Rp;
  for (int i = tid; i < ROWS * CH; i += 128) {
    const int r = i / CH, c = (i % CH) * 8;
    const bool ok = f0 + r < nf;
    cp_async16(sQ + r * LD + c, ok ? (const void*)(q + (long long)r * Rp + c) : (const void*)plane, ok);
  }
  auto fetch = [&](int pg, int buf) {
    const __nv_bfloat16* src = plane + (long long)tab[pg] * KV_PAGE * Rp;
    const int valid = min(KV_PAGE, p_hi + 1 - pg * KV_PAGE);       // keys beyond the tile's last position: zero
    for (int i = tid; i < KV_PAGE * CH; i += 128) {
      const int r = i / CH, c = (i % CH) * 8;
      const bool ok = r < valid;
      cp_async16(sC + (buf * KV_PAGE + r) * LD + c, ok ? (const void*)(src + (long long)r * Rp + c) : (const void*)plane, ok);
    }
    cp_async_commit();
  };
  float acc[MT][NT][4];
  float m_run[MT][2], l_run[MT][2];
#pragma unroll
  for (int i = 0; i < MT; ++i) {
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][j][e] = 0.f;
#pragma unroll
    for (int e = 0; e < 2; ++e) { m_run[i][e] = -CUDART_INF_F; l_run[i][e] = 0.f; }
  }
  // position of the rows this thread holds (rows lane / 4 and lane / 4 + 8 of every tile); -1 beyond the entry
  int rp[MT][2];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int f = f0 + 16 * i + (lane >> 2) + 8 * e;
      rp[i][e] = f < nf ? start + f / a.H : -1;
    }
  if (pg0 < pg1) fetch(pg0, 0); else cp_async_commit();
  for (int pg = pg0, buf = 0; pg < pg1; ++pg, buf ^= 1) {
    if (pg + 1 < pg1) { fetch(pg + 1, buf ^ 1); cp_async_wait<1>(); } else cp_async_wait<0>();
    __syncthreads();
    const __nv_bfloat16* C = sC + buf * KV_PAGE * LD;
    // scores: 16 MT rows x 16 keys per warp
    float s[MT][2][4];
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[i][j][e] = 0.f;
#pragma unroll 4
    for (int kk = 0; kk < Rp; kk += 16) {
      unsigned b0[2], b1[2];
      {
        const int r = warp * 16 + (lane & 7) + ((lane >> 4) << 3), c = kk + (((lane >> 3) & 1) << 3);
        ldmatrix_x4(b0[0], b0[1], b1[0], b1[1], C + r * LD + c);
      }
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        unsigned af[4];
        ldmatrix_x4(af[0], af[1], af[2], af[3], sQ + (16 * i + (lane & 15)) * LD + kk + ((lane >> 4) << 3));
        mma_bf16(s[i][0], af, b0);
        mma_bf16(s[i][1], af, b1);
      }
    }
    // mask, scale, row maxima of this warp's keys
    const int key0 = pg * KV_PAGE + warp * 16 + (lane & 3) * 2;
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        float mx = -CUDART_INF_F;
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            const int key = key0 + 8 * j + x, dist = rp[i][e] - key;
            const bool see = dist >= 0 && (a.window <= 0 || dist < a.window);
            float& v = s[i][j][2 * e + x];
            v = see ? v * a.scale : -CUDART_INF_F;
            mx = fmaxf(mx, v);
          }
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        if ((lane & 3) == 0) sMax[warp * ROWS + 16 * i + (lane >> 2) + 8 * e] = mx;
      }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = 16 * i + (lane >> 2) + 8 * e;
        float mx = m_run[i][e];
#pragma unroll
        for (int w = 0; w < 4; ++w) mx = fmaxf(mx, sMax[w * ROWS + r]);
        const float f = mx == -CUDART_INF_F ? 1.f : expf(m_run[i][e] - mx);
        m_run[i][e] = mx;
        float sum = 0.f;
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          float p0 = mx == -CUDART_INF_F ? 0.f : expf(s[i][j][2 * e] - mx), p1 = mx == -CUDART_INF_F ? 0.f : expf(s[i][j][2 * e + 1] - mx);
          sum += p0 + p1;
          *reinterpret_cast<__nv_bfloat162*>(sP + r * PLD + warp * 16 + 8 * j + (lane & 3) * 2) = __floats2bfloat162_rn(p0, p1);
        }
        sum += __shfl_xor_sync(0xffffffffu, sum, 1);
        sum += __shfl_xor_sync(0xffffffffu, sum, 2);
        if ((lane & 3) == 0) sSum[warp * ROWS + r] = sum;
        l_run[i][e] *= f;
#pragma unroll
        for (int j = 0; j < NT; ++j) { acc[i][j][2 * e] *= f; acc[i][j][2 * e + 1] *= f; }
      }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = 16 * i + (lane >> 2) + 8 * e;
#pragma unroll
        for (int w = 0; w < 4; ++w) l_run[i][e] += sSum[w * ROWS + r];
      }
    // output columns of this warp
#pragma unroll
    for (int kk = 0; kk < KV_PAGE; kk += 16) {
      unsigned af[MT][4];
#pragma unroll
      for (int i = 0; i < MT; ++i)
        ldmatrix_x4(af[i][0], af[i][1], af[i][2], af[i][3], sP + (16 * i + (lane & 15)) * PLD + kk + ((lane >> 4) << 3));
#pragma unroll
      for (int j = 0; j < NT; j += 2) {
        // keys kk .. kk + 15 (k) x 16 columns (n), stored row-major by key: transposed fragments.  With an odd NT the
        // last read covers eight columns of the next warp (or the pad), whose product is dropped
        unsigned b0[2], b1[2];
        const int r = kk + (lane & 7) + (((lane >> 3) & 1) << 3), c = warp * (Rp / 4) + 8 * j + ((lane >> 4) << 3);
        ldmatrix_x4_trans(b0[0], b0[1], b1[0], b1[1], C + r * LD + c);
#pragma unroll
        for (int i = 0; i < MT; ++i) {
          mma_bf16(acc[i][j], af[i], b0);
          if (j + 1 < NT) mma_bf16(acc[i][j + 1 < NT ? j + 1 : j], af[i], b1);
        }
      }
    }
    __syncthreads();
  }
  cp_async_wait<0>();
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int f = f0 + 16 * i + (lane >> 2) + 8 * e;
      if (f >= nf) continue;
      const long long rf = (long long)r0 * a.H + f;
      const int h = f % a.H, col = warp * (Rp / 4) + (lane & 3) * 2;
      if (a.splits > 1) {
        const long long pr = (long long)blockIdx.x * a.rows.M * a.H + rf;
#pragma unroll
        for (int j = 0; j < NT; ++j)
          *reinterpret_cast<float2*>(a.part_o + pr * Rp + col + 8 * j) = make_float2(acc[i][j][2 * e], acc[i][j][2 * e + 1]);
        if (warp == 0 && (lane & 3) == 0) { a.part_ml[2 * pr] = m_run[i][e]; a.part_ml[2 * pr + 1] = l_run[i][e]; }
        continue;
      }
      float m = m_run[i][e], l = l_run[i][e], w = 1.f;
      if (a.sink) {
        const float sk = a.sink[h], m2 = fmaxf(m, sk);
        w = expf(m - m2);
        l = l * w + expf(sk - m2);
      }
      w = w / l * (a.gate ? a.gate[rf] : 1.f);
      __nv_bfloat16* o = reinterpret_cast<__nv_bfloat16*>(a.out) + rf * Rp;
#pragma unroll
      for (int j = 0; j < NT; ++j)
        *reinterpret_cast<__nv_bfloat162*>(o + col + 8 * j) = __floats2bfloat162_rn(acc[i][j][2 * e] * w, acc[i][j][2 * e + 1] * w);
    }
}

// merges the key splits: one CTA of 128 threads per (row, head).  grid M H
template <typename T>
__global__ void __launch_bounds__(128) latent_merge_kernel(LatentArgs a) {
  __shared__ float s_w[32];
  const long long n = (long long)a.rows.M * a.H, rf = blockIdx.x;
  const int lane = threadIdx.x & 31;
  // every warp: lane s holds split s (at most 32)
  const float ms = lane < a.splits ? a.part_ml[2 * (lane * n + rf)] : -CUDART_INF_F;
  const float ls = lane < a.splits ? a.part_ml[2 * (lane * n + rf) + 1] : 0.f;
  const float sk = a.sink ? a.sink[rf % a.H] : -CUDART_INF_F;
  float m = fmaxf(ms, sk);
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
  const float f = expf(ms - m);
  const float l = warp_sum(ls * f) + (a.sink ? expf(sk - m) : 0.f);
  if (threadIdx.x < 32) s_w[lane] = f * ((a.gate ? a.gate[rf] : 1.f) / l);
  __syncthreads();
  for (int j = threadIdx.x * 4; j < a.Rp; j += 512) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int s = 0; s < a.splits; ++s) {
      const float4 t = *reinterpret_cast<const float4*>(a.part_o + (s * n + rf) * a.Rp + j);
      const float ws = s_w[s];
      v.x = fmaf(t.x, ws, v.x); v.y = fmaf(t.y, ws, v.y); v.z = fmaf(t.z, ws, v.z); v.w = fmaf(t.w, ws, v.w);
    }
    T* o = reinterpret_cast<T*>(a.out) + rf * a.Rp + j;
    o[0] = from_f<T>(v.x); o[1] = from_f<T>(v.y); o[2] = from_f<T>(v.z); o[3] = from_f<T>(v.w);
  }
}

// rows of a tile for an entry of f = tokens * heads rows
inline int latent_tile_rows(int Rp, int f) { return f <= 16 ? 16 : (f <= 32 || Rp > 256) ? 32 : 64; }
// attention (mma: the tensor-core kernel) and, with splits, the merge
int32_t vn_latent_attention(vn_ctx* ctx, const LatentArgs& a, bool bf16, bool mma);
