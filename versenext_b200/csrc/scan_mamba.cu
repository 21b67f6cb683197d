// Launches of the selective scan kernels.
#include "scan_mamba.cuh"

namespace {

template <typename T>
int32_t scan(vn_ctx* ctx, const MambaArgs& a) {
  const int ns = ceil_div(a.nstate, MAMBA_L);
  const dim3 grid(ceil_div(a.inner, MAMBA_CH), a.rows.n_ent);
#define SCAN(NS) VN_LAUNCH_NAMED(ctx, "mamba_scan_kernel", (mamba_scan_kernel<T, NS>), grid, 128, 0, a)
  if (ns <= 1) SCAN(1); else if (ns <= 2) SCAN(2); else if (ns <= 4) SCAN(4); else if (ns <= 6) SCAN(6);
  else if (ns <= 8) SCAN(8); else if (ns <= 16) SCAN(16); else SCAN(32);
#undef SCAN
  return VN_OK;
}

template <typename T>
int32_t step(vn_ctx* ctx, const MambaArgs& a) {
  const int ns = ceil_div(a.nstate, MAMBA_L);
  const dim3 grid(ceil_div(a.inner, 64), a.rows.M);
  const size_t smem = (size_t)(a.dt_cols + 2 * a.nstate) * 4;
#define STEP(NS) VN_LAUNCH_NAMED(ctx, "mamba_step_kernel", (mamba_step_kernel<T, NS>), grid, 256, smem, a)
  if (ns <= 1) STEP(1); else if (ns <= 2) STEP(2); else if (ns <= 4) STEP(4); else if (ns <= 6) STEP(6);
  else if (ns <= 8) STEP(8); else if (ns <= 16) STEP(16); else STEP(32);
#undef STEP
  return VN_OK;
}

}  // namespace

int32_t vn_mamba_scan(vn_ctx* ctx, const MambaArgs& a, bool bf16) {
  return bf16 ? scan<__nv_bfloat16>(ctx, a) : scan<float>(ctx, a);
}
int32_t vn_mamba_step(vn_ctx* ctx, const MambaArgs& a, bool bf16) {
  VN_REQUIRE(ctx, a.dt_cols + 2 * a.nstate <= 12000, "dt rank %d too large for the step kernel", a.dt_rank);
  return bf16 ? step<__nv_bfloat16>(ctx, a) : step<float>(ctx, a);
}
