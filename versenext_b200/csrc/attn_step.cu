// The one-token kernel of paged_attn.cuh.
//
// CTA = (key range, key/value head and tile of 16 query heads, sequence).  It convolves and rotates its query heads; the
// CTA of the last range does the same for the new key and value and appends them.  Each of four warps streams chunks of 16
// keys through its own cp.async ring; the warps, then the CTAs of a sequence (the last one to finish), merge.
#include "ldmatrix.cuh"
#include "paged_attn.cuh"

namespace {

using bf16 = __nv_bfloat16;
constexpr int WARPS = 4;
template <int P> constexpr int stages() { return P > 128 ? 2 : 3; }
template <int P> constexpr int step_smem() { return WARPS * stages<P>() * 2 * 16 * (P + 8) * 2 + 16 * (P + 8) * 2 + 2 * P * 2; }

// HEADS: biases, norms, interleaved pairs, factors of and caps on the scores, gates per head (an instance of its own: the code is fetched anew at every step)
template <int P, bool HEADS>
__global__ void __launch_bounds__(32 * WARPS, P > 128 ? 1 : 2) attn_step_kernel(ConvIn<bf16, Src, false> in, PagedAttnArgs a) {
  using namespace mma_detail;
  constexpr int LD = P + 8, ST = stages<P>(), TH = 32 * WARPS, CH = P / 8, TILE = 16 * LD;
  extern __shared__ __align__(16) unsigned char raw[];
  bf16* ring = reinterpret_cast<bf16*>(raw);                          // [warp][stage][K, V][16][LD]
  bf16* sQ = ring + WARPS * ST * 2 * TILE;                            // [16][LD]
  bf16* sNew = sQ + TILE;                                             // [2][P] key and value of the new token
  // convolved channels: query heads 0 .. 15, key (16), value (17); they lie in ring stages that no prefetch has reached yet
  auto sConv = [&](int r) { return reinterpret_cast<float*>(ring + ((r < 16 ? 0 : ST * 2) + (ST - 1) * 2) * TILE) + (r < 16 ? r : r - 16) * P; };
  __shared__ int s_last;
  __shared__ float s_ml[WARPS][16][2], s_f[WARPS][16], s_norm[17], s_gate[16];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, row = blockIdx.z;
  const int hg = a.H / a.KH, tiles = (hg + 15) / 16, g = blockIdx.y / tiles, q0 = (blockIdx.y % tiles) * 16, nq = min(16, hg - q0);
  int slot, r0, n, pos;
  a.rows.entry(a.rows.entry_of(row), &slot, &r0, &n, &pos);
  const int lo = a.first_key(pos);
  const int c_lo = lo / 16, c_hi = pos / 16 + 1, per = (c_hi - c_lo + a.splits - 1) / a.splits;
  const int c0 = min(c_hi, c_lo + (int)blockIdx.x * per), c1 = min(c_hi, c0 + per);
  const bool fresh = a.own_kv && c0 < c1 && c1 == c_hi;               // this range ends with the new token
  const int* tab = a.table + (long long)slot * a.max_pages;
  const long long ldp = (long long)a.KH * P;
  const bf16 *kp = reinterpret_cast<const bf16*>(a.kplane) + (long long)g * P, *vp = reinterpret_cast<const bf16*>(a.vplane) + (long long)g * P;
  bf16* mine = ring + warp * ST * 2 * TILE;
  auto fetch = [&](int c, int st) {
    if (c < c1) {
      const long long base = ((long long)tab[16 * c / KV_PAGE] * KV_PAGE + 16 * c % KV_PAGE) * ldp;
      const int valid = min(16, pos + (fresh ? 0 : 1) - 16 * c);      // the new token's row comes from shared memory
      for (int i = lane; i < 16 * CH; i += 32) {
        const int r = i / CH, x = (i % CH) * 8;
        const bool ok = r < valid;
        const long long at = base + (ok ? r : 0) * ldp + x;
        cp_async16(mine + st * 2 * TILE + r * LD + x, kp + at, ok);
        cp_async16(mine + st * 2 * TILE + TILE + r * LD + x, vp + at, ok);
      }
    }
    cp_async_commit();
  };
#pragma unroll
  for (int s = 0; s < ST - 1; ++s) fetch(c0 + warp + s * WARPS, s);
  if (tid < (a.rd / 2 + 15) / 16)                                     // the rotation's row is needed two barriers from here
    asm volatile("prefetch.global.L2 [%0];" ::"l"(a.rope + (long long)pos * (a.rd / 2) + 16 * tid));
  // queries; the new key and value
  {
    const int d = a.d, vd = a.vd, taps = in.taps, C = in.C, n_qk = (nq + (fresh ? 1 : 0)) * d, n_all = n_qk + (fresh ? vd : 0);
    // channel i of this CTA's list (query heads, key, value) -> column of the projection, place in sConv
    auto place = [&](int i, int& c, float*& dst, bool& keep) {
      const int head = i < n_qk ? i / d : nq + 1, x = i < n_qk ? i - head * d : i - n_qk;
      c = head < nq ? (g * hg + q0 + head) * d + x : head == nq ? (a.H + g) * d + x : (a.H + a.KH) * d + g * vd + x;
      dst = sConv(head < nq ? head : head == nq ? 16 : 17) + x;
      keep = head < nq ? blockIdx.x == 0 : q0 == 0;
    };
    bf16* inputs = in.ring + (long long)slot * in.RC * C;
    int c;
    float* dst;
    bool keep;
    if (d % 4 == 0 && vd % 4 == 0 && in.src.ld % 4 == 0 && C % 4 == 0 && taps <= 4) {
      // four channels at a time; one copy of the code, which is fetched anew at every step of a large model
#pragma unroll 1
      for (int i = tid * 4; i < n_all; i += TH * 4) {
        place(i, c, dst, keep);
        float4 x[4];
#pragma unroll
        for (int j = 1; j < 4; ++j) {
          x[j] = make_float4(0.f, 0.f, 0.f, 0.f);
          if (j < taps && j <= pos) x[j] = load4(inputs + (long long)((pos - j) % in.RC) * C + c);
        }
        x[0] = get4(in.src, row, c);
        if (keep && taps > 1) store4(inputs + (long long)(pos % in.RC) * C + c, x[0]);
        x[0] = make_float4(round_to<bf16>(x[0].x), round_to<bf16>(x[0].y), round_to<bf16>(x[0].z), round_to<bf16>(x[0].w));
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
        const float* w = in.w + (long long)c * taps + taps - 1;
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (j < taps) {
            acc.x = fmaf(x[j].x, w[-j], acc.x); acc.y = fmaf(x[j].y, w[taps - j], acc.y);
            acc.z = fmaf(x[j].z, w[2 * taps - j], acc.z); acc.w = fmaf(x[j].w, w[3 * taps - j], acc.w);
          }
        if (HEADS && in.bias) { const float4 b = load4(in.bias + c); acc.x += b.x; acc.y += b.y; acc.z += b.z; acc.w += b.w; }
        store4(dst, acc);
      }
    } else {
#pragma unroll 1
      for (int i = tid; i < n_all; i += TH) {
        place(i, c, dst, keep);
        float cur;
        *dst = in.at(row, r0, pos, slot, c, &cur);
        if (keep && taps > 1) in.keep(slot, pos, c, cur);
      }
    }
    __syncthreads();
    if (HEADS && a.qn) {                                              // factors of the heads' norms
#pragma unroll 1
      for (int head = warp; head < nq + (fresh ? 1 : 0); head += WARPS) {
        const float* src = sConv(head < nq ? head : 16);
        float ss = 0.f;
        for (int x = lane; x < d; x += 32) ss = fmaf(src[x], src[x], ss);
        ss = warp_sum(ss);
        if (lane == 0) s_norm[head] = 1.f / sqrtf(ss / (float)d + a.eps);
      }
      __syncthreads();
    }
    // rotation of the queries and the key
    const int np = a.rd / 2, half = np + d - a.rd;
    const float2* rope = a.rope + (long long)pos * np;
    if (HEADS && a.gate_head && tid < nq) s_gate[tid] = in.src.get_rare(row, a.col_g + g * hg + q0 + tid);
#pragma unroll 1
    for (int i = tid; i < (nq + (fresh ? 1 : 0)) * half; i += TH) {
      const int head = i / half, x = i - head * half;
      const float* src = sConv(head < nq ? head : 16);
      bf16* to = head < nq ? sQ + head * LD : sNew;
      const bool pair = x < np, next = HEADS && a.interleaved;
      const int cu = !pair ? np + x : next ? 2 * x : x, cv = !pair ? cu : next ? 2 * x + 1 : np + x;
      float fu = 1.f, fv = 1.f;
      if (HEADS && a.qn) {
        const float* nw = head < nq ? a.qn : a.kn;
        fu = s_norm[head] * nw[cu];
        fv = s_norm[head] * nw[cv];
      }
      if (HEADS && a.temp && head < nq) {
        const float t = a.temp[g * hg + q0 + head];
        fu *= t;
        fv *= t;
      }
      if (pair) {
        const float2 cs = rope[x];
        const float u = src[cu] * fu, v = src[cv] * fv;
        to[cu] = __float2bfloat16_rn(u * cs.x - v * cs.y);
        to[cv] = __float2bfloat16_rn(v * cs.x + u * cs.y);
      } else {
        to[cu] = __float2bfloat16_rn(src[cu] * fu);
      }
    }
    if (fresh)
      for (int x = tid; x < vd; x += TH) sNew[P + x] = __float2bfloat16_rn(sConv(17)[x]);
    const bf16 zero = __float2bfloat16_rn(0.f);
    for (int i = tid; i < 16 * P; i += TH) {
      const int r = i / P, c = i % P;
      if (r >= nq || c >= d) sQ[r * LD + c] = zero;
    }
    if (fresh) {
      for (int c = d + tid; c < P; c += TH) sNew[c] = zero;
      for (int c = vd + tid; c < P; c += TH) sNew[P + c] = zero;
    }
  }
  __syncthreads();
  if (fresh && q0 == 0) {
    const long long at = (((long long)tab[pos / KV_PAGE] * KV_PAGE + pos % KV_PAGE) * a.KH + g) * P;
    for (int c = tid; c < P; c += TH) {
      reinterpret_cast<bf16*>(a.kplane)[at + c] = sNew[c];
      reinterpret_cast<bf16*>(a.vplane)[at + c] = sNew[P + c];
    }
  }
  float acc[P / 8][4];
#pragma unroll
  for (int j = 0; j < P / 8; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
  float m_run[2] = {-CUDART_INF_F, -CUDART_INF_F}, l_run[2] = {0.f, 0.f};
  const bool capped = HEADS && a.softcap > 0.f;
  const float sc = capped ? 1.f : a.scale * 1.4426950408889634f;
  const bf16* q_at = sQ + (lane & 15) * LD + ((lane >> 4) << 3);
  int st = 0;
  for (int c = c0 + warp; c < c1; c += WARPS) {
    fetch(c + (ST - 1) * WARPS, st == 0 ? ST - 1 : st - 1);
    cp_async_wait<ST - 1>();
    __syncwarp();
    bf16 *K = mine + st * 2 * TILE, *V = K + TILE;
    if (fresh && c == pos / 16) {
      for (int x = lane; x < P; x += 32) { K[(pos & 15) * LD + x] = sNew[x]; V[(pos & 15) * LD + x] = sNew[P + x]; }
      __syncwarp();
    }
    float s[2][4];
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[j][e] = 0.f;
#pragma unroll
    for (int k = 0; k < P / 16; ++k) {
      unsigned af[4], b0[2], b1[2];
      ldmatrix_x4(af[0], af[1], af[2], af[3], q_at + 16 * k);
      ldmatrix_x4(b0[0], b0[1], b1[0], b1[1], K + ((lane & 7) + ((lane >> 4) << 3)) * LD + 16 * k + (((lane >> 3) & 1) << 3));
      mma_bf16(s[0], af, b0);
      mma_bf16(s[1], af, b1);
    }
    if (capped)
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int x = 0; x < 4; ++x) s[j][x] = softcap_log2(s[j][x] * a.scale, a.softcap);
    float mx[2] = {m_run[0], m_run[1]};
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int key = 16 * c + 8 * j + (lane & 3) * 2 + (x & 1);
        s[j][x] = key >= lo && key <= pos ? s[j][x] * sc : -CUDART_INF_F;
        mx[x >> 1] = fmaxf(mx[x >> 1], s[j][x]);
      }
    float f[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 1));
      mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 2));
      f[e] = exp2f(m_run[e] - mx[e]);                     // a chunk has a visible key, so mx is finite
      m_run[e] = mx[e];
      l_run[e] *= f[e];
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        s[j][x] = exp2f(s[j][x] - mx[x >> 1]);
        l_run[x >> 1] += s[j][x];
      }
    const unsigned af[4] = {pack_bf16(s[0][0], s[0][1]), pack_bf16(s[0][2], s[0][3]), pack_bf16(s[1][0], s[1][1]), pack_bf16(s[1][2], s[1][3])};
#pragma unroll
    for (int j = 0; j < P / 16; ++j) {
      unsigned b0[2], b1[2];
      ldmatrix_x4_t(b0[0], b0[1], b1[0], b1[1], V + ((lane & 7) + (((lane >> 3) & 1) << 3)) * LD + 16 * j + ((lane >> 4) << 3));
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        acc[2 * j + y][0] *= f[0]; acc[2 * j + y][1] *= f[0]; acc[2 * j + y][2] *= f[1]; acc[2 * j + y][3] *= f[1];
      }
      mma_bf16(acc[2 * j], af, b0);
      mma_bf16(acc[2 * j + 1], af, b1);
    }
    __syncwarp();
    st = st + 1 == ST ? 0 : st + 1;
  }
  cp_async_wait<0>();
  __syncthreads();                                        // the rings are free: outputs of the warps [warp][16][P]
  float* sO = reinterpret_cast<float*>(raw);
  static_assert(WARPS * 16 * P * 4 <= WARPS * ST * 2 * TILE * 2, "outputs fit where the rings were");
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    float l = l_run[e];
    l += __shfl_xor_sync(0xffffffffu, l, 1);
    l += __shfl_xor_sync(0xffffffffu, l, 2);
    const int r = (lane >> 2) + 8 * e;
    if ((lane & 3) == 0) { s_ml[warp][r][0] = m_run[e]; s_ml[warp][r][1] = l; }
#pragma unroll
    for (int j = 0; j < P / 8; ++j)
      *reinterpret_cast<float2*>(sO + (warp * 16 + r) * P + 8 * j + (lane & 3) * 2) = make_float2(acc[j][2 * e], acc[j][2 * e + 1]);
  }
  __syncthreads();
  // factors of the warps, and the range's own maximum and sum
  if (tid < 16) {
    float m = -CUDART_INF_F, l = 0.f;
#pragma unroll
    for (int w = 0; w < WARPS; ++w) m = fmaxf(m, s_ml[w][tid][0]);
#pragma unroll
    for (int w = 0; w < WARPS; ++w) {
      const float f = s_ml[w][tid][0] == -CUDART_INF_F ? 0.f : exp2f(s_ml[w][tid][0] - m);
      s_f[w][tid] = f;
      l += f * s_ml[w][tid][1];
    }
    s_ml[0][tid][0] = m;
    s_ml[0][tid][1] = l;
  }
  __syncthreads();
  // four columns of a head: divided by the sum, gated, stored
  const bool vec = a.vd % 4 == 0 && (a.gate_head || (a.col_g % 4 == 0 && in.src.ld % 4 == 0));
  auto gates = [&](int r, int c) {
    const int col = a.col_g + (g * hg + q0 + r) * a.vd + c;
    if (a.col_g < 0 || c >= a.vd) return make_float4(0.f, 0.f, 0.f, 0.f);
    if (HEADS && a.gate_head) return make_float4(s_gate[r], s_gate[r], s_gate[r], s_gate[r]);
    if (vec) return get4(in.src, row, col);
    const int last = a.vd - 1 - c;
    return make_float4(in.src.get_rare(row, col), in.src.get_rare(row, col + min(1, last)), in.src.get_rare(row, col + min(2, last)),
                       in.src.get_rare(row, col + min(3, last)));
  };
  auto finish = [&](int r, int c, float4 o, float l, float4 gt) {
    if (c >= a.vd) return;
    const float inv = 1.f / l;
    float v[4] = {o.x * inv, o.y * inv, o.z * inv, o.w * inv};
    if (a.col_g >= 0) { v[0] *= sigmoid_f(gt.x); v[1] *= sigmoid_f(gt.y); v[2] *= sigmoid_f(gt.z); v[3] *= sigmoid_f(gt.w); }
    bf16* out = reinterpret_cast<bf16*>(a.out) + ((long long)row * a.H + g * hg + q0 + r) * a.vd + c;
    if (vec) store4(out, make_float4(v[0], v[1], v[2], v[3]));
    else
      for (int e = 0; e < 4 && c + e < a.vd; ++e) out[e] = __float2bfloat16_rn(v[e]);
  };
  const long long n_rh = (long long)a.rows.M * a.H, rh0 = (long long)row * a.H + g * hg + q0;
#pragma unroll 1
  for (int i = tid; i < nq * (P / 4); i += TH) {
    const int r = i / (P / 4), c = i % (P / 4) * 4;
    float4 gt, o = make_float4(0.f, 0.f, 0.f, 0.f);
    if (a.splits == 1) gt = gates(r, c);
#pragma unroll
    for (int w = 0; w < WARPS; ++w) {
      const float4 t = load4(sO + (w * 16 + r) * P + c);
      const float f = s_f[w][r];
      o.x = fmaf(f, t.x, o.x); o.y = fmaf(f, t.y, o.y); o.z = fmaf(f, t.z, o.z); o.w = fmaf(f, t.w, o.w);
    }
    if (a.splits == 1) finish(r, c, o, s_ml[0][r][1], gt);
    else store4(a.part_o + ((long long)blockIdx.x * n_rh + rh0 + r) * P + c, o);
  }
  if (a.splits == 1) return;
  if (tid < nq) {
    float* ml = a.part_ml + ((long long)blockIdx.x * n_rh + rh0 + tid) * 2;
    ml[0] = s_ml[0][tid][0];
    ml[1] = s_ml[0][tid][1];
  }
  __threadfence();
  __syncthreads();
  if (tid == 0) {
    int* t = a.tickets + (long long)row * gridDim.y + blockIdx.y;
    s_last = atomicAdd(t, 1) == a.splits - 1;
    if (s_last) *t = 0;
  }
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  // merge the ranges: weight of range s for head r in shared memory (lane s holds range s), then the heads' sums
  float* sW = reinterpret_cast<float*>(raw);              // [32][16], then [16]
  for (int r = warp; r < nq; r += WARPS) {
    const float* ml = a.part_ml + ((long long)lane * n_rh + rh0 + r) * 2;
    const float m = lane < a.splits ? __ldcg(ml) : -CUDART_INF_F, l = lane < a.splits ? __ldcg(ml + 1) : 0.f;
    float top = m;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, o));
    const float f = m == -CUDART_INF_F ? 0.f : exp2f(m - top);
    const float sum = warp_sum(f * l);
    sW[lane * 16 + r] = f;
    if (lane == 0) sW[512 + r] = sum;
  }
  __syncthreads();
#pragma unroll 1
  for (int i = tid; i < nq * (P / 4); i += TH) {
    const int r = i / (P / 4), c = i % (P / 4) * 4;
    const float4 gt = gates(r, c);
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    const float* part = a.part_o + (rh0 + r) * P + c;
#pragma unroll 8
    for (int s = 0; s < a.splits; ++s) {
      const float4 t = __ldcg(reinterpret_cast<const float4*>(part + s * n_rh * P));
      const float f = sW[s * 16 + r];
      o.x = fmaf(f, t.x, o.x); o.y = fmaf(f, t.y, o.y); o.z = fmaf(f, t.z, o.z); o.w = fmaf(f, t.w, o.w);
    }
    finish(r, c, o, sW[512 + r], gt);
  }
}

}  // namespace

int32_t vn_attn_step(vn_ctx* ctx, const ConvIn<bf16, Src, false>& conv, const PagedAttnArgs& a) {
  const dim3 grid(a.splits, a.KH * ceil_div(a.H / a.KH, 16), a.rows.M);
  VN_REQUIRE(ctx, a.splits >= 1 && a.splits <= 32 && (a.splits == 1 || (long long)grid.y * grid.z <= VN_TICKETS), "key ranges of the one-token kernel");
  const bool heads = conv.bias || a.qn || a.interleaved || a.temp || a.gate_head || a.softcap > 0.f;
#define STEP1(P, HEADS) do { \
    static unsigned long long done = 0; \
    if (!((done >> (ctx->device & 63)) & 1ull)) { \
      VN_CUDA(ctx, cudaFuncSetAttribute((attn_step_kernel<P, HEADS>), cudaFuncAttributeMaxDynamicSharedMemorySize, step_smem<P>())); \
      done |= 1ull << (ctx->device & 63); \
    } \
    VN_LAUNCH_NAMED(ctx, "attn_step_kernel", (attn_step_kernel<P, HEADS>), grid, 32 * WARPS, step_smem<P>(), conv, a); } while (0)
#define STEP(P) do { if (heads) STEP1(P, true); else STEP1(P, false); } while (0)
  switch (a.P) {
    case 32: STEP(32); break;
    case 64: STEP(64); break;
    case 96: STEP(96); break;
    case 128: STEP(128); break;
    case 192: STEP(192); break;
    case 256: STEP(256); break;
    default: return vn_fail(ctx, VN_ERR_UNSUPPORTED, "key pitch %d", a.P);
  }
#undef STEP
#undef STEP1
  return VN_OK;
}
