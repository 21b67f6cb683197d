// Residual arrangements of composed models beyond x + f(norm(x)): several residual streams that are read as a weighted sum
// and mixed with one another at every write (hyper-connections), a gate on each sublayer's result, and a short causal
// convolution on what a mixer reads.  Streams, weights, norms and gates are fp32.
#pragma once
#include "rows.cuh"

constexpr int MAX_STREAMS = 8;

// One pass over a row: the sublayer's result y is scaled and gated, the streams are mixed and written, the next sublayer's
// weighted sum u is read off and normalised.  S: type of the y and gate sources (they may be split-K slices).
template <typename T, typename S>
struct StreamArgs {
  float* x = nullptr;              // [M][ns][D]
  const float* first = nullptr;    // [M][D] what every stream holds before its first write, or null: x
  int ns = 1, D = 0;
  S y, gate;                       // [M, D]; y.p null: nothing to write; gate.p null: no gate
  const float* gate_b = nullptr;   // [D] or null
  const float* ss = nullptr;       // [M][n_ss] partial sums of squares: y is divided by sqrt(sum / ss_count + eps); or null
  int n_ss = 0;
  float ss_count = 1.f;
  const float* mix = nullptr;      // [from][to], null: every stream keeps itself
  const float* out = nullptr;      // [to], null: ones
  const float* in = nullptr;       // [ns] weights of u, null: ones
  const float* norm_w = nullptr;   // null: no norm is wanted
  int layer_norm = 0;              // 1: mean subtracted; 0: root mean square
  float eps = 0.f;
  T* h = nullptr;                  // normalised rows, or null
  float* h32 = nullptr;            // the same in fp32, or null
  const int* pick = nullptr;       // row of block b: pick[b], or b * mul + add (only without y)
  int mul = 1, add = 0;
  // convolution of h, for batches in which every entry brings one row: hc = h + conv(h)
  T* hc = nullptr;
  T* ring = nullptr;
  const float* conv_w = nullptr;   // [D, taps]
  int RC = 1, taps = 1;
  Rows rows;
};

template <typename T, typename S> int32_t vn_streams(vn_ctx* ctx, const StreamArgs<T, S>& a, int n_rows);
// x [M][ns][D] -> sum of the streams [M][D]
int32_t vn_streams_sum(vn_ctx* ctx, const float* x, float* out, int M, int ns, int D);
// hc = h + conv(h), any batch; the entries' inputs are kept when they are at most `pending`
template <typename T> int32_t vn_input_conv(vn_ctx* ctx, const ConvIn<T, Mat<T>, false>& in, const Rows& rows, int pending, T* hc);
