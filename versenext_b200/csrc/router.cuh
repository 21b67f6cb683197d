// Mixture of experts: which experts a row goes to.  Scores are the soft-max over all router outputs, or the sigmoid of each;
// the choice may see a correction per expert and be limited to the best groups of neighbouring experts; the weights are the
// plain scores.  The last outputs may be identity experts, whose result is their input.  A further column of the router's
// product may hold the raw gate of an expert that serves every row; it may also take a row's last slot, as expert E.  Rows are then laid out expert by expert by the kernels that
// serve the other mixtures (mod_dispatch_kernel, or mod_offsets / mod_scatter / gather_sorted).
#pragma once
#include "rows.cuh"
#include <math_constants.h>

constexpr int ROUTE_WARPS = 8, MAX_CHOSEN = 32;
inline int route_rows(int M) { return M >= 2048 ? 2 : 1; }      // rows per warp: a block's counts are added up before they leave it
inline size_t route_smem(int E, int groups) { return ((size_t)ROUTE_WARPS * (2 * E + groups) + E + 1) * 4; }

struct RouteIn {
  Src z;                               // [M, E or more] router outputs
  int sigmoid = 0;                     // scores: sigmoid of each output, else soft-max over all
  const float* correction = nullptr;   // [E] or null
  int M = 0, E = 0, top = 1, groups = 1, keep = 1, rows = 1;      // rows: per warp
  int* slot_expert = nullptr;          // [M, top + shared_slot]
  float* slot_w = nullptr;             // as slot_expert
  int* count = nullptr;                // [E + shared_slot], zero before the launch
  float* shared_gate = nullptr;        // [M] sigmoid of column E, or null
  int shared_slot = 0;                 // slot `top` of every row is expert E with weight 1
};

// index of the largest value over a warp's lanes (the lowest one among equals), by way of integers in the same order
__device__ __forceinline__ int warp_argmax(float v, int i) {
  const unsigned bits = __float_as_uint(v), key = bits ^ ((bits >> 31) ? 0xffffffffu : 0x80000000u);
  const unsigned top = __reduce_max_sync(0xffffffffu, key);
  return (int)__reduce_min_sync(0xffffffffu, key == top ? (unsigned)i : 0xffffffffu);
}

// one warp per `rows` rows.  grid ceil(M / (ROUTE_WARPS rows)), shared memory route_smem
__global__ void __launch_bounds__(32 * ROUTE_WARPS) route_kernel(RouteIn r) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ float s_route[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, E = r.E;
  int* s_count = reinterpret_cast<int*>(s_route + ROUTE_WARPS * (2 * E + r.groups));
  const int n_count = E + r.shared_slot, slots = r.top + r.shared_slot;
  for (int e = threadIdx.x; e < n_count; e += 32 * ROUTE_WARPS) s_count[e] = 0;
  __syncthreads();
  const int first = (blockIdx.x * ROUTE_WARPS + warp) * r.rows;
#pragma unroll 1
  for (int row = first; row < min(r.M, first + r.rows); ++row) {
    float* score = s_route + warp * (2 * E + r.groups);
    float* choice = score + E;
    float* best = choice + E;
    float top = -CUDART_INF_F;
    for (int e = lane; e < E; e += 32) {
      const float z = r.z.get(row, e);
      score[e] = z;
      top = fmaxf(top, z);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, o));
    float sum = 0.f;
    if (!r.sigmoid)
      for (int e = lane; e < E; e += 32) { const float x = expf(score[e] - top); score[e] = x; sum += x; }
    sum = warp_sum(sum);
    if (r.shared_gate && lane == 0) {
      r.shared_gate[row] = sigmoid_f(r.z.get(row, E));
      if (r.shared_slot) {
        r.slot_expert[(long long)row * slots + r.top] = E;
        r.slot_w[(long long)row * slots + r.top] = 1.f;
        atomicAdd(s_count + E, 1);
      }
    }
    for (int e = lane; e < E; e += 32) {
      const float s = r.sigmoid ? sigmoid_f(score[e]) : score[e] / sum;
      score[e] = s;
      choice[e] = r.correction ? s + r.correction[e] : s;
    }
    __syncwarp();
    const int per = E / r.groups;
    if (r.keep < r.groups) {
      for (int g = lane; g < r.groups; g += 32) {
        float m = choice[g * per];
        for (int i = 1; i < per; ++i) m = fmaxf(m, choice[g * per + i]);
        best[g] = m;
      }
      __syncwarp();
      // the groups that are not kept: all but `keep` times the largest
      for (int k = 0; k < r.keep; ++k) {
        float v = -CUDART_INF_F;
        int at = r.groups;
        for (int g = lane; g < r.groups; g += 32)
          if (best[g] != CUDART_INF_F && (best[g] > v || at == r.groups)) { v = best[g]; at = g; }
        at = warp_argmax(v, at);
        if (lane == 0 && at < r.groups) best[at] = CUDART_INF_F;          // marks a kept group
        __syncwarp();
      }
      for (int e = lane; e < E; e += 32)
        if (best[e / per] != CUDART_INF_F) choice[e] = -CUDART_INF_F;
      __syncwarp();
    }
    for (int k = 0; k < r.top; ++k) {
      float v = -CUDART_INF_F;
      int at = E;
      for (int e = lane; e < E; e += 32)
        if (choice[e] > v) { v = choice[e]; at = e; }
      at = warp_argmax(v, at);
      if (lane == 0) {
        at = at < E ? at : 0;                                             // not finite scores: any expert
        r.slot_expert[(long long)row * slots + k] = at;
        r.slot_w[(long long)row * slots + k] = score[at];
        atomicAdd(s_count + at, 1);
        choice[at] = -CUDART_INF_F;
      }
      __syncwarp();
    }
  }
  __syncthreads();
  for (int e = threadIdx.x; e < n_count; e += 32 * ROUTE_WARPS)
    if (s_count[e]) atomicAdd(r.count + e, s_count[e]);
}
