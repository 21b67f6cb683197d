// Launches of the selective scan kernels.
#include "scan_mamba.cuh"

namespace {

template <typename T>
int32_t scan(vn_ctx* ctx, const MambaArgs& a) {
  const dim3 grid(ceil_div(a.inner, MAMBA_CH), a.rows.n_ent);
#define SCAN(NS, L) VN_LAUNCH_NAMED(ctx, "mamba_scan_kernel", (mamba_scan_kernel<T, NS, L>), grid, 32 * L, 0, a)
  // few sequences: eight lanes per channel, so that every scheduler has more than one warp
  if (a.nstate >= 8 && a.nstate <= 32 && (long long)grid.x * grid.y <= 2 * ctx->sm_count) {
    if (a.nstate <= 16) SCAN(2, 8); else SCAN(4, 8);
    return VN_OK;
  }
  const int ns = ceil_div(a.nstate, 4);
  if (ns <= 1) SCAN(1, 4); else if (ns <= 2) SCAN(2, 4); else if (ns <= 4) SCAN(4, 4); else if (ns <= 6) SCAN(6, 4);
  else if (ns <= 8) SCAN(8, 4); else if (ns <= 16) SCAN(16, 4); else SCAN(32, 4);
#undef SCAN
  return VN_OK;
}

template <typename T>
int32_t step(vn_ctx* ctx, const MambaArgs& a) {
  const size_t smem = (size_t)(a.dt_cols + 2 * a.nstate) * 4;
#define STEP(NS, L) VN_LAUNCH_NAMED(ctx, "mamba_step_kernel", (mamba_step_kernel<T, NS, L>), \
                                    dim3(ceil_div(a.inner, 256 / L), a.rows.M), 256, smem, a)
  const int n = a.nstate;
  if (n <= 4) STEP(2, 2); else if (n <= 8) STEP(4, 2); else if (n <= 16) STEP(8, 2); else if (n <= 24) STEP(6, 4);
  else if (n <= 32) STEP(8, 4); else if (n <= 64) STEP(16, 4); else STEP(32, 4);
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
