// Launches of the gated delta rule kernels.
#include "scan_delta.cuh"

template <typename T>
int32_t vn_delta_inputs(vn_ctx* ctx, const ConvIn<T>& conv, const DeltaIn& in) {
  const dim3 grid(2 * in.KH + in.H + 1, ceil_div(in.rows.M, 8)), block(32, 8);
  const int nc = ceil_div(in.d > in.vd ? in.d : in.vd, 32);
#define INPUTS(NC) VN_LAUNCH_NAMED(ctx, "delta_inputs_kernel", (delta_inputs_kernel<T, NC>), grid, block, 0, conv, in)
  if (nc <= 1) INPUTS(1); else if (nc <= 2) INPUTS(2); else if (nc <= 4) INPUTS(4); else if (nc <= 8) INPUTS(8); else INPUTS(16);
#undef INPUTS
  return VN_OK;
}
template int32_t vn_delta_inputs<float>(vn_ctx*, const ConvIn<float>&, const DeltaIn&);
template int32_t vn_delta_inputs<__nv_bfloat16>(vn_ctx*, const ConvIn<__nv_bfloat16>&, const DeltaIn&);

template <typename T>
int32_t vn_delta_step(vn_ctx* ctx, const DeltaStepArgs<T>& a) {
  const dim3 grid(a.in.H, a.in.rows.M);
  const int d = a.in.d;
  const int extra = 2 * a.in.vd + a.in.ra_ld + a.in.rg_ld;
  VN_REQUIRE(ctx, extra + 24 * 32 <= 12000, "low-rank factors too wide for the step kernel");
#define STEP(DK) VN_LAUNCH_NAMED(ctx, "delta_step_kernel", (delta_step_kernel<T, DK>), grid, 256, (size_t)(24 * DK + extra) * 4, a)
  if (d <= 32) STEP(4); else if (d <= 64) STEP(8); else if (d <= 96) STEP(12); else if (d <= 128) STEP(16); else STEP(32);
#undef STEP
  return VN_OK;
}
template int32_t vn_delta_step<float>(vn_ctx*, const DeltaStepArgs<float>&);
template int32_t vn_delta_step<__nv_bfloat16>(vn_ctx*, const DeltaStepArgs<__nv_bfloat16>&);

int32_t vn_delta_scan(vn_ctx* ctx, const DeltaRuleArgs& a) {
  const dim3 grid(ceil_div(a.vd, DR_COLS), a.H, a.rows.n_ent);
  const int d = a.d;
  const bool vec = d % 4 == 0 && a.vd % 4 == 0;
#define SCAN(DK) do { if (vec) VN_LAUNCH_NAMED(ctx, "delta_scan_kernel", (delta_scan_kernel<DK, 4>), grid, 128, 0, a); \
                      else VN_LAUNCH_NAMED(ctx, "delta_scan_kernel", (delta_scan_kernel<DK, 1>), grid, 128, 0, a); } while (0)
  if (d <= 32) SCAN(4); else if (d <= 64) SCAN(8); else if (d <= 96) SCAN(12); else if (d <= 128) SCAN(16); else SCAN(32);
#undef SCAN
  return VN_OK;
}
