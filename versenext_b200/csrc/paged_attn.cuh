// Grouped-query attention over paged keys and values: query head h reads key/value head h / (H / KH).  Optional sliding
// window or chunks, rotary positions on the first rd dimensions of a head (half-split or interleaved pairs; frequencies and
// amplitude come as a table), biases, an RMS norm of every query and key head, short causal convolutions on q, k and v, a
// factor of every query head's scores, a soft cap of the scores, a sigmoid gate on every output element or every head; scores
// and soft-max in fp32.  A layer may read another layer's planes instead of owning some.
//
// Cache: plane[page * KV_PAGE + pos % KV_PAGE][KH][P], P = padded width of a key or value; table[slot * max_pages + pos / KV_PAGE].
#pragma once
#include "gemm_mma.cuh"
#include "rows.cuh"
#include <math_constants.h>

struct PagedAttnArgs {
  int H = 0, KH = 0, d = 0, vd = 0, P = 0;
  int window = 0;                  // position i sees j with 0 <= i - j < window; 0: no limit
  int chunk = 0;                   // position i sees no j before the last multiple of chunk; 0: no limit
  float scale = 1.f, softcap = 0.f;   // softcap c > 0: a score s becomes c tanh(s / c)
  const float* qn = nullptr;       // [d] weights of the query heads' and key heads' norms, or null
  const float* kn = nullptr;
  float eps = 0.f;
  const float* temp = nullptr;     // [H] factors of the scores (the queries are stored times them), or null
  int rd = 0;                      // rotated dimensions (even)
  int interleaved = 0;             // dimension 2 i is rotated with 2 i + 1, else i with i + rd / 2
  const float2* rope = nullptr;    // [positions][rd / 2] cos, sin
  int own_kv = 1;                  // 0: the planes belong to another layer and hold this step's rows already
  void* kplane = nullptr; void* vplane = nullptr;
  const int* table = nullptr;
  int max_pages = 0;
  int col_g = -1;                  // first gate column of the projection, or -1
  int gate_head = 0;               // gates: one per head, else one per output element
  void* q = nullptr;               // [M, H, P] storage dtype
  void* out = nullptr;             // [M, H vd] storage dtype
  // one-token kernel: key ranges of a sequence, merged by the CTA that finishes last
  int splits = 1;                  // at most 32
  float* part_o = nullptr;         // [splits][M * H][P] unnormalised
  float* part_ml = nullptr;        // [splits][M * H][2]
  int* tickets = nullptr;          // zero between kernels
  int pending = 1;
  Rows rows;
  // the first key that position pos sees
  __device__ __forceinline__ int first_key(int pos) const {
    const int lo = window > 0 ? max(0, pos - window + 1) : 0;
    return chunk > 0 ? max(lo, pos - pos % chunk) : lo;
  }
};

// c tanh(s / c) times log2(e), for exp2f: tanh(x) = 1 - 2 / (exp(2 x) + 1)
__device__ __forceinline__ float softcap_log2(float s, float cap) {
  const float c2 = cap * 1.4426950408889634f;
  return c2 - __fdividef(2.f * c2, exp2f(s * (2.885390081777927f / cap)) + 1.f);
}

// convolution, or bias and norm, and rotation of q and k, the same of v; keys and values to their pages
template <typename T, typename S> int32_t vn_attn_inputs(vn_ctx* ctx, const ConvIn<T, S, false>& conv, const PagedAttnArgs& a);
// attention of all rows behind vn_attn_inputs; mma: the tensor-core kernel
template <typename T, typename S> int32_t vn_paged_attention(vn_ctx* ctx, const S& proj, const PagedAttnArgs& a, bool mma);
// one new row per sequence: everything between the two projections
int32_t vn_attn_step(vn_ctx* ctx, const ConvIn<__nv_bfloat16, Src, false>& conv, const PagedAttnArgs& a);
// cos and sin of positions 0 .. rows - 1, times amp
int32_t vn_rope_table(vn_ctx* ctx, const double* freq_dev, int pairs, float amp, int rows, float2* out);
// padded width of a key or value that the tensor-core kernels have an instance for, else a multiple of 32
inline int attn_pitch(int w) {
  for (int t : {32, 64, 96, 128, 192, 256})
    if (w <= t) return t;
  return (w + 31) & ~31;
}
inline bool attn_mma_ok(int P) { return P <= 256; }
