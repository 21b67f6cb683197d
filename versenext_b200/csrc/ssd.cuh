// State-space duality (Mamba-2): per head a state S [N, P] in fp32 with one decay per token,
//
//   S <- exp(A dt) S + dt B x^T ;  y = S^T C + D x ;  u = y silu(z) ,
//
// dt = softplus(projection + bias), x, B and C from a short causal convolution with silu, B and C shared by the heads of a
// group.  u is then normed in equal parts over all heads (ssd_norm) and multiplied by a weight.
//
// Projection columns: z [H P] | x [H P] | B [G N] | C [G N] | dt [H].  State layout [slot][R][head][P][N] (a column of S is
// contiguous); ring of states as in scan_mamba.cuh.
#pragma once
#include "gemm_mma.cuh"
#include "rows.cuh"

struct SsdArgs {
  int H = 0, P = 0, N = 0, G = 1;
  void* xbc = nullptr;             // [M, ld] convolved and activated x | B | C, storage dtype
  int ld = 0;
  float* dt = nullptr;             // [M, H] step sizes
  void* z = nullptr;               // [M, H P] the gates in the storage dtype, or null: read off the projection (see vn_ssd_scan)
  const float* dt_bias = nullptr;  // [H]
  const float* A = nullptr;        // [H] -exp(A_log)
  const float* D = nullptr;        // [H]
  float* state = nullptr;
  int R = 2, pending = 1;
  void* u = nullptr;               // [M, H P] storage dtype
  // workspace of the chunked kernel with several segments: [n_ent][segments][H][P][N], what the segments but the last add to
  // the state, then the state that the entry starts with (its place in the ring may be the one the last segment writes);
  // [n_ent][segments][H] the segments' decays (as exponents of 2)
  float* seg_state = nullptr;
  float* seg_decay = nullptr;
  int segments = 1, seg_len = 0;   // pieces of the entries that run at once; rows of each (a multiple of 64)
  Rows rows;
  __host__ __device__ int inner() const { return H * P; }
  __host__ __device__ int channels() const { return H * P + 2 * G * N; }
  __host__ __device__ int col_dt() const { return 2 * H * P + 2 * G * N; }
};

// how a forward of these rows runs, and the workspace
struct SsdPlan { bool chunked = false; int segments = 1, seg_len = 0; size_t seg_bytes = 0; };
SsdPlan vn_ssd_plan(const vn_ctx* ctx, bool bf16, int H, int N, int P, const Rows& rows, int pending);

// convolution of x, B and C, step sizes (everything but the one-token kernel needs them)
template <typename T, typename S> int32_t vn_ssd_inputs(vn_ctx* ctx, const ConvIn<T, S>& conv, const SsdArgs& a);
// token after token (all entries of one row: a kernel of its own, which reads z when the projection is Src): any dtype, any count; the states behind all tokens are kept when there are fewer than R
template <typename T, typename S> int32_t vn_ssd_scan(vn_ctx* ctx, const S& proj, const SsdArgs& a);
// chunks of 64 tokens on the tensor cores (N <= 128)
template <typename S> int32_t vn_ssd_chunks(vn_ctx* ctx, const S& proj, const SsdArgs& a);
constexpr int SSD_STEP_ROWS = 16;
// one new row per sequence, few of them: convolution, step size, recurrence and gate
template <typename T> int32_t vn_ssd_step(vn_ctx* ctx, const ConvIn<T>& conv, const SsdArgs& a);
// out = u over the root mean square of its part (`parts` equal ones) times w
template <typename T> int32_t vn_ssd_norm(vn_ctx* ctx, const T* u, const float* w, T* out, int M, int n, int parts, float eps);
