// Lightning attention: a linear attention whose state decays by one constant per head, S [dim, vdim] in fp32,
//
//   S <- decay S + k v^T ; o = S^T q ,   q, k, v = silu of their projections
//
// followed by a norm over all heads' outputs together, a weight and a sigmoid gate.  The norm's factor is one number per
// row, so these kernels write o * weight * gate and the row's partial sums of squares, and whoever adds the output
// projection to the residual stream divides by the root mean square.
//
// State layout [slot][R][head][vdim][dim] (a column is contiguous); ring of states as in scan_mamba.cuh.
#pragma once
#include "gemm_mma.cuh"
#include "rows.cuh"

struct LightningArgs {
  int H = 0, d = 0, vd = 0;
  int activated = 0;               // 1: q, k, v columns of the source went through silu already
  const float* decay = nullptr;    // [H][2] the constant as a sum of two floats
  const float* powers = nullptr;   // [H][65] its powers 0 .. 64
  const float* norm_w = nullptr;   // [H vd]
  float* state = nullptr;
  int R = 2;
  void* out = nullptr;             // [M, H vd] storage dtype
  float* ss = nullptr;             // [M, n_ss] partial sums of squares of o
  int n_ss = 0;                    // see LightningPlan
  // workspace of the chunked kernel with several segments, [n_ent][segments][H][vd][d]: what the segments but the last add
  // to the state, then the state that the entry starts with (its place in the ring may be the one the last segment writes)
  float* seg_state = nullptr;
  int segments = 1, seg_len = 0;   // pieces of the entries that run at once; rows of each (a multiple of 64)
  Rows rows;
};

// how a forward of these rows runs; fixes n_ss and the workspace
struct LightningPlan { bool chunked = false; int n_ss = 1, segments = 1, seg_len = 0; size_t seg_bytes = 0; };
LightningPlan vn_lightning_plan(const vn_ctx* ctx, bool bf16, int H, int d, int vd, const Rows& rows, int pending);

// token after token: any dtype, any count; the states behind all tokens are kept when there are fewer than R
template <typename T, typename S> int32_t vn_lightning_scan(vn_ctx* ctx, const S& proj, const LightningArgs& a);
// chunks of 64 tokens on the tensor cores; source activated and in bf16
int32_t vn_lightning_chunks(vn_ctx* ctx, const Mat<__nv_bfloat16>& proj, const LightningArgs& a);
