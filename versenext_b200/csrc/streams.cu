// Kernels of streams.cuh.
#include "streams.cuh"

namespace {

template <int V> struct Vec { float v[V]; };
template <int V, typename P> __device__ __forceinline__ Vec<V> vload(const P* p) {
  Vec<V> r;
  if constexpr (V == 4) { const float4 t = load4(p); r.v[0] = t.x; r.v[1] = t.y; r.v[2] = t.z; r.v[3] = t.w; }
  else r.v[0] = to_f(*p);
  return r;
}
template <int V, typename S> __device__ __forceinline__ Vec<V> vget(const S& s, long long row, int d) {
  Vec<V> r;
  if constexpr (V == 4) { const float4 t = get4(s, row, d); r.v[0] = t.x; r.v[1] = t.y; r.v[2] = t.z; r.v[3] = t.w; }
  else r.v[0] = s.get(row, d);
  return r;
}
template <int V, typename P> __device__ __forceinline__ void vstore(P* p, const Vec<V>& r) {
  if constexpr (V == 4) store4(p, make_float4(r.v[0], r.v[1], r.v[2], r.v[3]));
  else *p = from_f<P>(r.v[0]);
}

// One CTA per row.  Shared memory: D floats (u).
template <typename T, typename S, int NS, int V>
__global__ void __launch_bounds__(256) streams_kernel(StreamArgs<T, S> a) {
  pdl_trigger();
  extern __shared__ __align__(16) float s_u[];
  __shared__ float s_mix[NS * NS], s_out[NS], s_in[NS], red[3][8];
  const int tid = threadIdx.x, D = a.D;
  if (tid < NS * NS) s_mix[tid] = a.mix ? a.mix[tid] : (tid / NS == tid % NS ? 1.f : 0.f);
  if (tid < NS) { s_out[tid] = a.out ? a.out[tid] : 1.f; s_in[tid] = a.in ? a.in[tid] : 1.f; }
  pdl_wait();
  const long long row = a.pick ? a.pick[blockIdx.x] : (long long)blockIdx.x * a.mul + a.add;
  const bool write = a.y.p != nullptr, gated = a.gate.p != nullptr;
  float ysc = 1.f;
  if (a.ss) {
    float v = 0.f;
    for (int i = tid; i < a.n_ss; i += 256) v += a.ss[row * a.n_ss + i];
    ysc = 1.f / sqrtf(block_sum256(v, red[0]) / a.ss_count + a.eps);   // the sum's barrier also publishes the weights
  } else {
    __syncthreads();
  }
  float* x = a.x + row * NS * D;
  const float* first = a.first ? a.first + row * D : nullptr;
  float sum = 0.f;
  for (int d = tid * V; d < D; d += 256 * V) {
    Vec<V> xs[NS], u;
    if (first) {
      xs[0] = vload<V>(first + d);
#pragma unroll
      for (int s = 1; s < NS; ++s) xs[s] = xs[0];
    } else {
#pragma unroll
      for (int s = 0; s < NS; ++s) xs[s] = vload<V>(x + (long long)s * D + d);
    }
    if (write) {
      Vec<V> y = vget<V>(a.y, row, d), n[NS];
      if (gated) {
        const Vec<V> g = vget<V>(a.gate, row, d);
#pragma unroll
        for (int e = 0; e < V; ++e) y.v[e] *= sigmoid_f(g.v[e] + (a.gate_b ? a.gate_b[d + e] : 0.f));
      }
#pragma unroll
      for (int t = 0; t < NS; ++t) {
#pragma unroll
        for (int e = 0; e < V; ++e) {
          float v = s_out[t] * (y.v[e] * ysc);
#pragma unroll
          for (int s = 0; s < NS; ++s) v = fmaf(s_mix[s * NS + t], xs[s].v[e], v);
          n[t].v[e] = v;
        }
        vstore<V>(x + (long long)t * D + d, n[t]);
      }
#pragma unroll
      for (int t = 0; t < NS; ++t) xs[t] = n[t];
    }
#pragma unroll
    for (int e = 0; e < V; ++e) {
      u.v[e] = 0.f;
#pragma unroll
      for (int s = 0; s < NS; ++s) u.v[e] = fmaf(s_in[s], xs[s].v[e], u.v[e]);
      sum += a.layer_norm ? u.v[e] : u.v[e] * u.v[e];
    }
    vstore<V>(s_u + d, u);
  }
  if (!a.norm_w) return;
  float mean = 0.f, r;
  const float tot = block_sum256(sum, red[1]);
  if (a.layer_norm) {
    mean = tot / (float)D;
    float v = 0.f;
    for (int d = tid * V; d < D; d += 256 * V)
#pragma unroll
      for (int e = 0; e < V; ++e) { const float t = s_u[d + e] - mean; v = fmaf(t, t, v); }
    r = sqrtf(block_sum256(v, red[2]) / (float)D + a.eps);
  } else {
    r = sqrtf(tot / (float)D + a.eps);
  }
  int slot = 0, r0, n, pos = 0;
  if (a.hc) a.rows.entry(a.rows.entry_of((int)row), &slot, &r0, &n, &pos);
  const long long orow = blockIdx.x;
  for (int d = tid * V; d < D; d += 256 * V) {
    Vec<V> v = vload<V>(s_u + d);
    const Vec<V> w = vload<V>(a.norm_w + d);
#pragma unroll
    for (int e = 0; e < V; ++e) v.v[e] = (v.v[e] - mean) / r * w.v[e];
    if (a.h) vstore<V>(a.h + orow * D + d, v);
    if (a.h32) vstore<V>(a.h32 + orow * D + d, v);
    if (a.hc) {
      T* ring = a.ring + (long long)slot * a.RC * D + d;
      Vec<V> acc;
#pragma unroll
      for (int e = 0; e < V; ++e) {
        v.v[e] = round_to<T>(v.v[e]);
        acc.v[e] = v.v[e] * a.conv_w[(long long)(d + e) * a.taps + a.taps - 1];
      }
#pragma unroll 3
      for (int j = 1; j < a.taps; ++j) {
        if (j > pos) break;
        const Vec<V> old = vload<V>(ring + (long long)((pos - j) % a.RC) * D);
#pragma unroll
        for (int e = 0; e < V; ++e) acc.v[e] = fmaf(old.v[e], a.conv_w[(long long)(d + e) * a.taps + a.taps - 1 - j], acc.v[e]);
      }
      if (a.taps > 1) vstore<V>(ring + (long long)(pos % a.RC) * D, v);
#pragma unroll
      for (int e = 0; e < V; ++e) acc.v[e] += v.v[e];
      vstore<V>(a.hc + orow * D + d, acc);
    }
  }
}

// The same for few rows and D <= 2048 (a multiple of 4): a thread keeps its four columns of everything in registers, so that
// all loads are in flight together; weights are fetched ahead of the wait on the preceding kernel; one block reduction, of
// counts, means and squared deviations.  D / 4 threads, rounded up to whole warps.
struct Moments { float n, mean, m2; };
__device__ __forceinline__ Moments merge(const Moments& a, const Moments& b) {
  const float n = a.n + b.n;
  if (n == 0.f) return a;
  const float d = b.mean - a.mean, f = b.n / n;
  return {n, fmaf(d, f, a.mean), a.m2 + b.m2 + d * d * a.n * f};
}

template <typename T, typename S, int NS>
__global__ void __launch_bounds__(512) streams_row_kernel(StreamArgs<T, S> a) {
  pdl_trigger();
  __shared__ float s_mix[NS * NS], s_out[NS], s_in[NS];
  __shared__ Moments s_mom[16];
  const int tid = threadIdx.x, lane = tid & 31, D = a.D, d = tid * 4;
  const bool on = d < D;
  if (tid < NS * NS) s_mix[tid] = a.mix ? a.mix[tid] : (tid / NS == tid % NS ? 1.f : 0.f);
  if (tid < NS) { s_out[tid] = a.out ? a.out[tid] : 1.f; s_in[tid] = a.in ? a.in[tid] : 1.f; }
  const float4 zero4 = make_float4(0.f, 0.f, 0.f, 0.f);
  const float4 wn = on && a.norm_w ? load4(a.norm_w + d) : zero4, gb = on && a.gate_b ? load4(a.gate_b + d) : zero4;
  float4 cw[4] = {zero4, zero4, zero4, zero4};              // filter of channel d + e, the current token's tap last
  const int taps = a.hc ? a.taps : 0;
  if (on && taps == 4) {
#pragma unroll
    for (int e = 0; e < 4; ++e) cw[e] = load4(a.conv_w + (long long)(d + e) * 4);
  }
  __syncthreads();
  pdl_wait();
  const long long row = a.pick ? a.pick[blockIdx.x] : (long long)blockIdx.x * a.mul + a.add;
  const bool write = a.y.p != nullptr, gated = a.gate.p != nullptr;
  int slot = 0, r0, n, pos = 0;
  if (a.hc) a.rows.entry(a.rows.entry_of((int)row), &slot, &r0, &n, &pos);
  float* x = a.x + row * NS * D + d;
  float4 xs[NS], y = zero4;
  float ysc = 1.f;
  if (on) {
    if (a.first) {
      xs[0] = load4(a.first + row * D + d);
#pragma unroll
      for (int s = 1; s < NS; ++s) xs[s] = xs[0];
    } else {
#pragma unroll
      for (int s = 0; s < NS; ++s) xs[s] = load4(x + (long long)s * D);
    }
    if (write) y = get4(a.y, row, d);
    if (write && gated) {
      const float4 g = get4(a.gate, row, d);
      y.x *= sigmoid_f(g.x + gb.x); y.y *= sigmoid_f(g.y + gb.y); y.z *= sigmoid_f(g.z + gb.z); y.w *= sigmoid_f(g.w + gb.w);
    }
  }
  if (a.ss) {                                               // every warp sums the row's parts
    float v = 0.f;
    for (int i = lane; i < a.n_ss; i += 32) v += a.ss[row * a.n_ss + i];
    ysc = 1.f / sqrtf(warp_sum(v) / a.ss_count + a.eps);
  }
  float4 u = zero4;
  if (on) {
    if (write) {
      y.x *= ysc; y.y *= ysc; y.z *= ysc; y.w *= ysc;
      float4 nx[NS];
#pragma unroll
      for (int t = 0; t < NS; ++t) {
        const float o = s_out[t];
        nx[t] = make_float4(o * y.x, o * y.y, o * y.z, o * y.w);
#pragma unroll
        for (int s = 0; s < NS; ++s) {
          const float m = s_mix[s * NS + t];
          nx[t].x = fmaf(m, xs[s].x, nx[t].x); nx[t].y = fmaf(m, xs[s].y, nx[t].y);
          nx[t].z = fmaf(m, xs[s].z, nx[t].z); nx[t].w = fmaf(m, xs[s].w, nx[t].w);
        }
        store4(x + (long long)t * D, nx[t]);
      }
#pragma unroll
      for (int t = 0; t < NS; ++t) xs[t] = nx[t];
    }
#pragma unroll
    for (int s = 0; s < NS; ++s) {
      const float m = s_in[s];
      u.x = fmaf(m, xs[s].x, u.x); u.y = fmaf(m, xs[s].y, u.y); u.z = fmaf(m, xs[s].z, u.z); u.w = fmaf(m, xs[s].w, u.w);
    }
  }
  if (!a.norm_w) return;
  Moments mo = {0.f, 0.f, 0.f};
  if (on) {
    if (a.layer_norm) {
      const float mean = (u.x + u.y + u.z + u.w) * 0.25f, p = u.x - mean, q = u.y - mean, v = u.z - mean, w = u.w - mean;
      mo = {4.f, mean, p * p + q * q + v * v + w * w};
    } else {
      mo = {4.f, 0.f, u.x * u.x + u.y * u.y + u.z * u.z + u.w * u.w};
    }
  }
#pragma unroll
  for (int o = 1; o < 32; o <<= 1)
    mo = merge(mo, {__shfl_xor_sync(0xffffffffu, mo.n, o), __shfl_xor_sync(0xffffffffu, mo.mean, o), __shfl_xor_sync(0xffffffffu, mo.m2, o)});
  if (lane == 0) s_mom[tid >> 5] = mo;
  __syncthreads();
  mo = s_mom[0];
  for (int w = 1; w < (int)blockDim.x / 32; ++w) mo = merge(mo, s_mom[w]);
  if (!on) return;
  const float r = sqrtf(mo.m2 / (float)D + a.eps);
  float v[4] = {(u.x - mo.mean) / r * wn.x, (u.y - mo.mean) / r * wn.y, (u.z - mo.mean) / r * wn.z, (u.w - mo.mean) / r * wn.w};
  const long long at = (long long)blockIdx.x * D + d;
  if (a.h) store4(a.h + at, make_float4(v[0], v[1], v[2], v[3]));
  if (a.h32) store4(a.h32 + at, make_float4(v[0], v[1], v[2], v[3]));
  if (!a.hc) return;
  T* ring = a.ring + (long long)slot * a.RC * D + d;
  float acc[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) v[e] = round_to<T>(v[e]);
  if (taps == 4) {
    float4 old[3] = {zero4, zero4, zero4};
#pragma unroll
    for (int j = 1; j < 4; ++j)
      if (j <= pos) old[j - 1] = load4(ring + (long long)((pos - j) % a.RC) * D);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      auto of = [&](const float4& t) { return e == 0 ? t.x : e == 1 ? t.y : e == 2 ? t.z : t.w; };
      acc[e] = fmaf(of(old[2]), cw[e].x, fmaf(of(old[1]), cw[e].y, fmaf(of(old[0]), cw[e].z, v[e] * cw[e].w)));
    }
  } else {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float* w = a.conv_w + (long long)(d + e) * taps;
      acc[e] = v[e] * w[taps - 1];
      for (int j = 1; j < taps && j <= pos; ++j) acc[e] = fmaf(to_f<T>(ring[(long long)((pos - j) % a.RC) * D + e]), w[taps - 1 - j], acc[e]);
    }
  }
  if (taps > 1) store4(ring + (long long)(pos % a.RC) * D, make_float4(v[0], v[1], v[2], v[3]));
  store4(a.hc + at, make_float4(v[0] + acc[0], v[1] + acc[1], v[2] + acc[2], v[3] + acc[3]));
}

__global__ void __launch_bounds__(256) streams_sum_kernel(const float* __restrict__ x, float* __restrict__ out, int ns, int D) {
  const long long row = blockIdx.x;
  for (int d = threadIdx.x; d < D; d += 256) {
    float v = 0.f;
    for (int s = 0; s < ns; ++s) v += x[(row * ns + s) * D + d];
    out[row * D + d] = v;
  }
}

// RB rows of one channel per thread (RB > 1: filters of at most four taps).  grid (ceil(D / 256), ceil(M / RB))
template <typename T, int RB>
__global__ void __launch_bounds__(256) input_conv_kernel(ConvIn<T, Mat<T>, false> in, Rows rows, int pending, T* __restrict__ hc) {
  const int c = blockIdx.x * 256 + threadIdx.x, D = in.C;
  if (c >= D) return;
  int row = blockIdx.y * RB;
  const int last = min(row + RB, rows.M);
  while (row < last) {                                  // stretches of one entry
    int slot, r0, n, start;
    rows.entry(rows.entry_of(row), &slot, &r0, &n, &start);
    const int end = min(last, r0 + n);
    float v[RB];
    if constexpr (RB > 1) {
      in.template run<RB>(row, end, r0, start, slot, c, v);
    } else {
      float cur;
      v[0] = in.at(row, r0, start, slot, c, &cur);
    }
#pragma unroll
    for (int i = 0; i < RB; ++i)
      if (row + i < end) {
        const float h = in.src.get(row + i, c);
        hc[(long long)(row + i) * D + c] = from_f<T>(h + v[i]);
        if (n <= pending && in.taps > 1) in.keep(slot, start + row + i - r0, c, h);
      }
    row = end;
  }
}

// four channels per thread, `rep` times RB rows, filters of at most four taps.  grid (ceil(D / 1024), ceil(M / (rep RB)))
template <typename T, int RB>
__global__ void __launch_bounds__(256) input_conv4_kernel(ConvIn<T, Mat<T>, false> in, Rows rows, int pending, int rep, T* __restrict__ hc) {
  const int c = (blockIdx.x * 256 + threadIdx.x) * 4, D = in.C;
  if (c >= D) return;
  int row = blockIdx.y * rep * RB;
  const int last = min(row + rep * RB, rows.M);
  float wt[4][4];
  in.filters4(c, wt);
#pragma unroll 1
  while (row < last) {                                  // stretches of one entry
    int slot, r0, n, start;
    rows.entry(rows.entry_of(row), &slot, &r0, &n, &start);
    const int end = min(min(last, row + RB), r0 + n);
    float4 v[RB];
    in.template run4<RB>(row, end, r0, start, slot, c, wt, v);
#pragma unroll
    for (int i = 0; i < RB; ++i)
      if (row + i < end) {
        const float4 h = load4(in.src.p + (long long)(row + i) * in.src.ld + c);
        store4(hc + (long long)(row + i) * D + c, make_float4(h.x + v[i].x, h.y + v[i].y, h.z + v[i].z, h.w + v[i].w));
        if (n <= pending && in.taps > 1) {
          const int pos = start + row + i - r0;
          in.keep(slot, pos, c, h.x); in.keep(slot, pos, c + 1, h.y); in.keep(slot, pos, c + 2, h.z); in.keep(slot, pos, c + 3, h.w);
        }
      }
    row = end;
  }
}

template <typename T, typename S, int V>
int32_t launch(vn_ctx* ctx, const StreamArgs<T, S>& a, int n_rows) {
  const size_t smem = (size_t)a.D * 4;
  const bool few = V == 4 && a.D <= 2048 && n_rows <= 1024;
  const int block = (a.D / 4 + 31) & ~31;
#define CASE(NS) case NS: \
  if constexpr (V == 4) { \
    if (few) { VN_LAUNCH_PDL_LEVEL(ctx, (vn_pdl_mask() & 4) ? 1 : 2, "streams_row_kernel", (streams_row_kernel<T, S, NS>), n_rows, block, 0, a); break; } \
  } \
  if (smem > 40000) VN_CUDA(ctx, cudaFuncSetAttribute((streams_kernel<T, S, NS, V>), cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
  VN_LAUNCH_PDL_LEVEL(ctx, (vn_pdl_mask() & 4) ? 1 : 2, "streams_kernel", (streams_kernel<T, S, NS, V>), n_rows, 256, smem, a); break;
  switch (a.ns) {
    CASE(1) CASE(2) CASE(3) CASE(4) CASE(5) CASE(6) CASE(7) CASE(8)
    default: return vn_fail(ctx, VN_ERR_UNSUPPORTED, "%d residual streams", a.ns);
  }
#undef CASE
  return VN_OK;
}

}  // namespace

template <typename T, typename S>
int32_t vn_streams(vn_ctx* ctx, const StreamArgs<T, S>& a, int n_rows) {
  if (a.D % 4 == 0 && a.y.ld % 4 == 0 && a.gate.ld % 4 == 0 && ((uintptr_t)a.gate.p & 15) == 0) return launch<T, S, 4>(ctx, a, n_rows);
  return launch<T, S, 1>(ctx, a, n_rows);
}
template int32_t vn_streams(vn_ctx*, const StreamArgs<float, Src>&, int);
template int32_t vn_streams(vn_ctx*, const StreamArgs<__nv_bfloat16, Src>&, int);
template int32_t vn_streams(vn_ctx*, const StreamArgs<__nv_bfloat16, Mat<__nv_bfloat16>>&, int);

int32_t vn_streams_sum(vn_ctx* ctx, const float* x, float* out, int M, int ns, int D) {
  VN_LAUNCH(ctx, streams_sum_kernel, M, 256, 0, x, out, ns, D);
  return VN_OK;
}

template <typename T>
int32_t vn_input_conv(vn_ctx* ctx, const ConvIn<T, Mat<T>, false>& in, const Rows& rows, int pending, T* hc) {
  const int rep = rows.M >= 2048 ? 2 : 1;
  if (in.taps <= 4 && in.C % 4 == 0)
    VN_LAUNCH_NAMED(ctx, "input_conv_kernel", (input_conv4_kernel<T, 8>), dim3(ceil_div(in.C, 1024), ceil_div(rows.M, 8 * rep)), 256, 0, in,
                    rows, pending, rep, hc);
  else if (in.taps <= 4)
    VN_LAUNCH_NAMED(ctx, "input_conv_kernel", (input_conv_kernel<T, 8>), dim3(ceil_div(in.C, 256), ceil_div(rows.M, 8)), 256, 0, in, rows,
                    pending, hc);
  else
    VN_LAUNCH_NAMED(ctx, "input_conv_kernel", (input_conv_kernel<T, 1>), dim3(ceil_div(in.C, 256), rows.M), 256, 0, in, rows, pending, hc);
  return VN_OK;
}
template int32_t vn_input_conv(vn_ctx*, const ConvIn<float, Mat<float>, false>&, const Rows&, int, float*);
template int32_t vn_input_conv(vn_ctx*, const ConvIn<__nv_bfloat16, Mat<__nv_bfloat16>, false>&, const Rows&, int, __nv_bfloat16*);
