// Kernels of lightning.cuh.
#include <algorithm>

#include "ldmatrix.cuh"
#include "lightning.cuh"
#include "scan_delta.cuh"      // columns of a state in registers

namespace {

using bf16 = __nv_bfloat16;
constexpr int SCAN_TH = 256, SCAN_COLS = SCAN_TH / 8;

// Eight lanes share a column; DK rows of it per lane (d <= 8 DK), NP columns per group.  A CTA runs over all rows of an
// entry with its columns in registers.  grid (H * ceil(vd / (32 NP)), n_ent)
template <typename T, typename S, int DK, int NP>
__global__ void __launch_bounds__(SCAN_TH) lightning_scan_kernel(LightningArgs a, S proj) {
  constexpr int DP = 8 * DK, COLS = SCAN_COLS * NP;
  __shared__ __align__(16) float s_q[2][DP], s_k[2][DP];
  __shared__ float s_v[2][COLS], red[2][SCAN_TH / 32];
  const int tid = threadIdx.x, nb = (a.vd + COLS - 1) / COLS, h = blockIdx.x / nb, cb = (blockIdx.x % nb) * COLS;
  const int d = a.d, vd = a.vd, cl = tid >> 3, li = tid & 7;
  int slot, r0, n, start;
  a.rows.entry(blockIdx.y, &slot, &r0, &n, &start);
  if (n <= 0) return;
  const long long one = (long long)vd * d;
  const float* st_in = a.state + (((long long)slot * a.R + start % a.R) * a.H + h) * one;
  float St[NP][DK];
#pragma unroll
  for (int p = 0; p < NP; ++p) {
    const int c = cb + cl + SCAN_COLS * p;
    delta_col_load<DK>(st_in + (long long)c * d, d, li, start > 0 && c < vd, St[p]);
  }
  const float dec = a.decay[2 * h], dec_lo = a.decay[2 * h + 1];
  const bool snap = n <= a.R - 1;
  const int kq = a.H * d, kv = 2 * a.H * d, kg = kv + a.H * vd, nv = min(COLS, vd - cb);
  for (int j = d + tid; j < DP; j += SCAN_TH) s_q[0][j] = s_q[1][j] = s_k[0][j] = s_k[1][j] = 0.f;
#pragma unroll 1
  for (int t = 0; t < n; ++t) {
    const int buf = t & 1;
    const long long row = r0 + t;
#pragma unroll 1
    for (int i = tid; i < 2 * d + nv; i += SCAN_TH) {
      const int c = i < d ? h * d + i : i < 2 * d ? kq + h * d + i - d : kv + h * vd + cb + i - 2 * d;
      float x = proj.get(row, c);
      if (!a.activated) x = round_to<T>(silu_as<T>(x));
      float* dst = i < d ? &s_q[buf][i] : i < 2 * d ? &s_k[buf][i - d] : &s_v[buf][i - 2 * d];
      *dst = x;
    }
    __syncthreads();
    float o[NP], v[NP];
#pragma unroll
    for (int p = 0; p < NP; ++p) { o[p] = 0.f; v[p] = cl + SCAN_COLS * p < nv ? s_v[buf][cl + SCAN_COLS * p] : 0.f; }
#pragma unroll
    for (int i = 0; i < DK / 4; ++i) {
      const float4 k4 = load4(&s_k[buf][32 * i + 4 * li]), q4 = load4(&s_q[buf][32 * i + 4 * li]);
      const float kk[4] = {k4.x, k4.y, k4.z, k4.w}, qq[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
      for (int p = 0; p < NP; ++p)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          float& s = St[p][4 * i + e];
          s = fmaf(dec, s, fmaf(dec_lo, s, kk[e] * v[p]));
          o[p] = fmaf(s, qq[e], o[p]);
        }
    }
    // lane p of a group finishes column p: weight, gate, output
    float mine = 0.f;
#pragma unroll
    for (int p = 0; p < NP; ++p) {
      o[p] += __shfl_xor_sync(0xffffffffu, o[p], 1);
      o[p] += __shfl_xor_sync(0xffffffffu, o[p], 2);
      o[p] += __shfl_xor_sync(0xffffffffu, o[p], 4);
      if (li == p) mine = o[p];
    }
    float ss = 0.f;
    const int cm = cl + SCAN_COLS * li;
    if (li < NP && cm < nv) {
      const int col = h * vd + cb + cm;
      ss = mine * mine;
      reinterpret_cast<T*>(a.out)[row * a.H * vd + col] = from_f<T>(mine * a.norm_w[col] * sigmoid_f(proj.get(row, kg + col)));
    }
    if (snap || t == n - 1) {
      float* st = a.state + (((long long)slot * a.R + (start + t + 1) % a.R) * a.H + h) * one;
#pragma unroll
      for (int p = 0; p < NP; ++p) {
        const int c = cb + cl + SCAN_COLS * p;
        if (c < vd) delta_col_store<DK>(st + (long long)c * d, d, li, St[p]);
      }
    }
    ss = warp_sum(ss);
    if ((tid & 31) == 0) red[buf][tid >> 5] = ss;
    __syncthreads();
    if (tid == 0) {
      float tot = 0.f;
#pragma unroll
      for (int i = 0; i < SCAN_TH / 32; ++i) tot += red[buf][i];
      a.ss[row * a.n_ss + blockIdx.x] = tot;
    }
  }
}

// columns per group: more fetch q and k fewer times, fewer make more CTAs
int scan_np(const vn_ctx* ctx, int H, int vd, int d, int n_ent) {
  if (d > 128) return 1;
  for (int np : {4, 2})
    if (vd > SCAN_COLS * np / 2 && (long long)n_ent * H * ceil_div(vd, SCAN_COLS * np) >= 2 * ctx->sm_count) return np;
  return 1;
}

// ---- chunked kernel ------------------------------------------------------------------------------------------------------
// A chunk of C tokens is three products: o = (lambda^(i+1) q_i) S + sum_{j <= i} lambda^(i-j) (q_i . k_j) v_j, and
// S <- lambda^C S + sum_j lambda^(C-1-j) k_j v_j^T.  q, k and v are 16-bit values; what is fp32 by nature (the state, the
// decayed scores, the decayed values) enters a tensor-core product as three bf16 pieces that add up to it, so nothing of
// the recurrence is computed at less than fp32.
//
// CTA = four warps, 64 columns of v of one head; warp w keeps the state of columns 16 w .. 16 w + 15 transposed in its
// accumulators [vd 16][d], which is also the layout its pieces have as the B operand of q S.
constexpr int CH = 64, CW = 4, VB = 16 * CW;

template <int DT> constexpr int chunk_smem(bool local) {
  const int q = 2 * CH * (DT + 8) * 2, v = 2 * CH * (VB + 8) * 2, p = CH * (CH + 4) * 4;
  return local ? q + v : 2 * q + v + p;
}

// LOCAL: only the state a segment would end with if it began with nothing, to seg_state (all but the last segment).
// grid (H * ceil(vd / VB), segments, n_ent)
template <int DT, bool LOCAL, bool VEC>
__global__ void __launch_bounds__(32 * CW) lightning_chunk_kernel(LightningArgs a, Mat<bf16> proj) {
  using namespace mma_detail;
  constexpr int LQ = DT + 8, LV = VB + 8, LP = CH + 4, TH = 32 * CW, NT = DT / 8;
  extern __shared__ __align__(16) unsigned char raw[];
  bf16* sK = reinterpret_cast<bf16*>(raw);                       // [2][CH][LQ]
  bf16* sV = sK + 2 * CH * LQ;                                   // [2][CH][LV]
  bf16* sQ = sV + 2 * CH * LV;                                   // [2][CH][LQ]
  float* sP = reinterpret_cast<float*>(sQ + (LOCAL ? 0 : 2 * CH * LQ));   // [CH][LP]
  __shared__ float s_pow[CH + 1];
  int slot, r0, n, start;
  a.rows.entry(blockIdx.z, &slot, &r0, &n, &start);
  const int seg = blockIdx.y, t_lo = seg * a.seg_len, t_hi = min(n, t_lo + a.seg_len);
  if (t_lo >= n) return;
  if (LOCAL && t_hi == n) return;                                // nobody starts behind the last piece
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int nvb = (a.vd + VB - 1) / VB, h = blockIdx.x / nvb, cb = (blockIdx.x % nvb) * VB, d = a.d, vd = a.vd;
  const int nv = min(VB, vd - cb), kq = a.H * d, kv = 2 * a.H * d, kg = kv + a.H * vd;
  if (tid <= CH) s_pow[tid] = a.powers[h * (CH + 1) + tid];
  // zero what no fetch writes: channels beyond d and columns beyond vd
  for (int i = tid; i < 2 * CH * (DT - d); i += TH) {
    const int r = i / (DT - d), c = d + i % (DT - d);
    sK[r * LQ + c] = __float2bfloat16_rn(0.f);
    if (!LOCAL) sQ[r * LQ + c] = __float2bfloat16_rn(0.f);
  }
  for (int i = tid; i < 2 * CH * (VB - nv); i += TH) sV[(i / (VB - nv)) * LV + nv + i % (VB - nv)] = __float2bfloat16_rn(0.f);
  auto fetch = [&](int t0, int buf) {
    const int m = min(CH, t_hi - t0);
    const bf16* base = proj.p + (long long)(r0 + t0) * proj.ld;
    if (VEC) {
      const int pd = d / 8, pv = nv / 8;
      for (int i = tid; i < CH * pd; i += TH) {
        const int r = i / pd, c = (i % pd) * 8;
        const bf16* src = base + (long long)(r < m ? r : 0) * proj.ld + h * d + c;
        if (!LOCAL) cp_async16(sQ + (buf * CH + r) * LQ + c, src, r < m);
        cp_async16(sK + (buf * CH + r) * LQ + c, src + kq, r < m);
      }
      for (int i = tid; i < CH * pv; i += TH) {
        const int r = i / pv, c = (i % pv) * 8;
        cp_async16(sV + (buf * CH + r) * LV + c, base + (long long)(r < m ? r : 0) * proj.ld + kv + h * vd + cb + c, r < m);
      }
    } else {
      const bf16 zero = __float2bfloat16_rn(0.f);
      for (int i = tid; i < CH * d; i += TH) {
        const int r = i / d, c = i % d;
        const bf16* src = base + (long long)r * proj.ld + h * d + c;
        if (!LOCAL) sQ[(buf * CH + r) * LQ + c] = r < m ? *src : zero;
        sK[(buf * CH + r) * LQ + c] = r < m ? src[kq] : zero;
      }
      for (int i = tid; i < CH * nv; i += TH) {
        const int r = i / nv, c = i % nv;
        sV[(buf * CH + r) * LV + c] = r < m ? base[(long long)r * proj.ld + kv + h * vd + cb + c] : zero;
      }
    }
    cp_async_commit();
  };
  fetch(t_lo, 0);
  // S[j][0..1]: column cb + 16 warp + lane / 4, rows 8 j + 2 (lane % 4) + {0, 1}; [2..3]: column + 8
  const int g4 = lane >> 2, l2 = (lane & 3) * 2;
  const long long one = (long long)vd * d;
  float S[NT][4];
  auto load_state = [&](const float* st, float keep) {           // S = keep S + st (keep 0: S = st)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int c = cb + 16 * warp + g4 + 8 * e;
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const int r = 8 * j + l2 + x;
          const float v = st && c < vd && r < d ? st[(long long)c * d + r] : 0.f;
          S[j][2 * e + x] = keep == 0.f ? v : fmaf(keep, S[j][2 * e + x], v);
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
          if (c < vd && r < d) st[(long long)c * d + r] = S[j][2 * e + x];
        }
    }
  };
  auto piece = [&](int s) { return a.seg_state + (((long long)blockIdx.z * a.segments + s) * a.H + h) * one; };
  const float* initial = start > 0 ? a.state + (((long long)slot * a.R + start % a.R) * a.H + h) * one : nullptr;
  if (LOCAL) {
    if (seg == 0 && initial) {
      load_state(initial, 0.f);
      store_state(piece(a.segments - 1));
    }
    load_state(nullptr, 0.f);
  } else {
    load_state(initial && n > a.seg_len ? piece(a.segments - 1) : initial, 0.f);
    if (seg > 0) {
      float keep = 1.f;                                          // decay over a whole piece
      const float full = a.powers[h * (CH + 1) + CH];
      for (int i = 0; i < a.seg_len / CH; ++i) keep *= full;
      keep = fmaxf(keep, 1e-38f);                                // 0 would mean "replace"
#pragma unroll 1
      for (int s = 0; s < seg; ++s) load_state(piece(s), keep);
    }
  }
  float nw[2][2];                                                // norm weights of the columns this lane finishes
#pragma unroll
  for (int j = 0; j < 2; ++j)
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int c = 16 * warp + 8 * j + l2 + x;
      nw[j][x] = !LOCAL && c < nv ? a.norm_w[h * vd + cb + c] : 0.f;
    }
#pragma unroll 1
  for (int t0 = t_lo, buf = 0; t0 < t_hi; t0 += CH, buf ^= 1) {
    unsigned gate[LOCAL || !VEC ? 1 : 4][2][2];                  // raw gates of this lane's outputs: requested ahead of the products
    if (!LOCAL && VEC)
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int e = 0; e < 2; ++e)
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const int t = t0 + 16 * i + g4 + 8 * e, c = 16 * warp + 8 * j + l2;
            if (t < t_hi && c < nv)
              gate[LOCAL || !VEC ? 0 : i][e][j] = *reinterpret_cast<const unsigned*>(proj.p + (long long)(r0 + t) * proj.ld + kg + h * vd + cb + c);
          }
    if (t0 + CH < t_hi) { fetch(t0 + CH, buf ^ 1); cp_async_wait<1>(); } else cp_async_wait<0>();
    __syncthreads();
    const int m = min(CH, t_hi - t0);
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
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          if (j > 2 * warp + 1) continue;
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int i = 16 * warp + g4 + 8 * e, c = 8 * j + l2;
            const float w0 = c <= i ? s_pow[max(i - c, 0)] : 0.f, w1 = c + 1 <= i ? s_pow[max(i - c - 1, 0)] : 0.f;
            *reinterpret_cast<float2*>(sP + i * LP + c) = make_float2(p[j][2 * e] * w0, p[j][2 * e + 1] * w1);
          }
        }
      }
      // q S, then the rows' decay
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
            split2(S[2 * k][2 * e], S[2 * k][2 * e + 1], b0[e]);
            split2(S[2 * k + 1][2 * e], S[2 * k + 1][2 * e + 1], b1[e]);
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
          const float w0 = s_pow[16 * i + g4 + 1], w1 = s_pow[16 * i + g4 + 9];
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
      // o * weight * gate, and the row's share of the sum of squares
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int t = 16 * i + g4 + 8 * e;
          const long long row = r0 + t0 + t;
          float ss = 0.f;
          if (t < m) {
#pragma unroll
            for (int j = 0; j < 2; ++j) {
              const int c = 16 * warp + 8 * j + l2;
              float v[2];
              float2 gv = make_float2(0.f, 0.f);
              if (VEC) gv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&gate[LOCAL || !VEC ? 0 : i][e][j]));
#pragma unroll
              for (int x = 0; x < 2; ++x) {
                v[x] = o[i][j][2 * e + x];
                ss = fmaf(v[x], v[x], ss);
                if (c + x < nv) {
                  const int col = h * vd + cb + c + x;
                  v[x] *= nw[j][x] * sigmoid_f(VEC ? (x ? gv.y : gv.x) : proj.get(row, kg + col));
                  if (!VEC) reinterpret_cast<bf16*>(a.out)[row * a.H * vd + col] = __float2bfloat16_rn(v[x]);
                }
              }
              if (VEC && c < nv)
                *reinterpret_cast<__nv_bfloat162*>(reinterpret_cast<bf16*>(a.out) + row * a.H * vd + h * vd + cb + c) = __floats2bfloat162_rn(v[0], v[1]);
            }
          }
          ss += __shfl_xor_sync(0xffffffffu, ss, 1);
          ss += __shfl_xor_sync(0xffffffffu, ss, 2);
          if (t < m && (lane & 3) == 0) a.ss[row * a.n_ss + blockIdx.x * CW + warp] = ss;
        }
    }
    // the state behind the chunk
    {
      const float all = s_pow[m];
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[j][e] *= all;
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        unsigned ar[4], ap[4][PIECES];
        ldmatrix_x4_t(ar[0], ar[1], ar[2], ar[3], V + (16 * k + (lane & 7) + ((lane >> 4) << 3)) * LV + 16 * warp + (((lane >> 3) & 1) << 3));
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const int t = 16 * k + l2 + 8 * (x >> 1);
          const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&ar[x]));
          split2(t < m ? f.x * s_pow[max(m - 1 - t, 0)] : 0.f, t + 1 < m ? f.y * s_pow[max(m - 2 - t, 0)] : 0.f, ap[x]);
        }
#pragma unroll
        for (int j = 0; j < DT / 16; ++j) {
          unsigned b0[2], b1[2];
          ldmatrix_x4_t(b0[0], b0[1], b1[0], b1[1], K + (16 * k + (lane & 7) + (((lane >> 3) & 1) << 3)) * LQ + 16 * j + ((lane >> 4) << 3));
#pragma unroll
          for (int x = PIECES - 1; x >= 0; --x) {
            const unsigned af[4] = {ap[0][x], ap[1][x], ap[2][x], ap[3][x]};
            mma_bf16(S[2 * j], af, b0);
            mma_bf16(S[2 * j + 1], af, b1);
          }
        }
      }
    }
    __syncthreads();
  }
  if (!LOCAL && t_hi < n) return;                                // only the last piece ends with the entry's state
  store_state(LOCAL ? piece(seg) : a.state + (((long long)slot * a.R + (start + n) % a.R) * a.H + h) * one);
}

template <int DT, bool VEC>
int32_t launch_chunks(vn_ctx* ctx, const Mat<bf16>& proj, const LightningArgs& a) {
  static unsigned long long done = 0;
  if (!((done >> (ctx->device & 63)) & 1ull)) {
    VN_CUDA(ctx, cudaFuncSetAttribute((lightning_chunk_kernel<DT, false, VEC>), cudaFuncAttributeMaxDynamicSharedMemorySize, chunk_smem<DT>(false)));
    VN_CUDA(ctx, cudaFuncSetAttribute((lightning_chunk_kernel<DT, true, VEC>), cudaFuncAttributeMaxDynamicSharedMemorySize, chunk_smem<DT>(true)));
    done |= 1ull << (ctx->device & 63);
  }
  const int gx = a.H * ceil_div(a.vd, VB);
  if (a.segments > 1)
    VN_LAUNCH_NAMED(ctx, "lightning_segment_kernel", (lightning_chunk_kernel<DT, true, VEC>), dim3(gx, a.segments - 1, a.rows.n_ent), 32 * CW,
                    chunk_smem<DT>(true), a, proj);
  VN_LAUNCH_NAMED(ctx, "lightning_chunk_kernel", (lightning_chunk_kernel<DT, false, VEC>), dim3(gx, a.segments, a.rows.n_ent), 32 * CW,
                  chunk_smem<DT>(false), a, proj);
  return VN_OK;
}

}  // namespace

LightningPlan vn_lightning_plan(const vn_ctx* ctx, bool bf16, int H, int d, int vd, const Rows& rows, int pending) {
  LightningPlan p;
  // few rows go token by token; so do rows that may be cut back (every state is kept), which only uniform batches have
  p.chunked = bf16 && d <= 128 && rows.max_n >= 8 && rows.max_n > pending;
  if (!p.chunked) {
    p.n_ss = H * ceil_div(vd, SCAN_COLS * scan_np(ctx, H, vd, d, rows.n_ent));
    return p;
  }
  const int nvb = ceil_div(vd, VB);
  p.n_ss = H * nvb * CW;
  const long long ctas = (long long)H * nvb * rows.n_ent;
  int s = (int)std::min<long long>(8, 2 * ctx->sm_count / std::max(1ll, ctas));
  s = std::max(1, std::min(s, rows.max_n / (4 * CH)));
  p.seg_len = ceil_div(ceil_div(rows.max_n, s), CH) * CH;
  p.segments = ceil_div(rows.max_n, p.seg_len);
  if (p.segments > 1) p.seg_bytes = (size_t)rows.n_ent * p.segments * H * d * vd * 4;
  return p;
}

template <typename T, typename S>
int32_t vn_lightning_scan(vn_ctx* ctx, const S& proj, const LightningArgs& a) {
  const int np = scan_np(ctx, a.H, a.vd, a.d, a.rows.n_ent);
  const dim3 grid(a.H * ceil_div(a.vd, SCAN_COLS * np), a.rows.n_ent);
#define SCAN2(DK, NP) VN_LAUNCH_NAMED(ctx, "lightning_scan_kernel", (lightning_scan_kernel<T, S, DK, NP>), grid, SCAN_TH, 0, a, proj)
#define SCAN(DK) do { if (np == 4) SCAN2(DK, 4); else if (np == 2) SCAN2(DK, 2); else SCAN2(DK, 1); } while (0)
  if (a.d <= 32) SCAN(4); else if (a.d <= 64) SCAN(8); else if (a.d <= 96) SCAN(12); else if (a.d <= 128) SCAN(16);
  else if (a.d <= 256) SCAN2(32, 1); else SCAN2(64, 1);
#undef SCAN
#undef SCAN2
  return VN_OK;
}
template int32_t vn_lightning_scan<float, Src>(vn_ctx*, const Src&, const LightningArgs&);
template int32_t vn_lightning_scan<bf16, Src>(vn_ctx*, const Src&, const LightningArgs&);
template int32_t vn_lightning_scan<bf16, Mat<bf16>>(vn_ctx*, const Mat<bf16>&, const LightningArgs&);

int32_t vn_lightning_chunks(vn_ctx* ctx, const Mat<bf16>& proj, const LightningArgs& a) {
  const bool vec = a.d % 8 == 0 && a.vd % 8 == 0 && proj.ld % 8 == 0 && ((uintptr_t)proj.p & 15) == 0;
#define CHUNKS(DT) return vec ? launch_chunks<DT, true>(ctx, proj, a) : launch_chunks<DT, false>(ctx, proj, a)
  if (a.d <= 32) CHUNKS(32);
  if (a.d <= 64) CHUNKS(64);
  if (a.d <= 96) CHUNKS(96);
  if (a.d <= 128) CHUNKS(128);
#undef CHUNKS
  return vn_fail(ctx, VN_ERR_UNSUPPORTED, "head width %d", a.d);
}
