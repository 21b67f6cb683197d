// Launches of the gated delta rule kernels.
#include "scan_delta.cuh"

template <typename T>
int32_t vn_delta_inputs(vn_ctx* ctx, const ConvIn<T>& conv, const DeltaIn& in) {
  const int nc = ceil_div(in.d > in.vd ? in.d : in.vd, 32);
  const bool many = in.rows.M >= 512 && nc <= 4 && conv.taps <= 4;
  const dim3 grid(2 * in.KH + in.H + 1, ceil_div(in.rows.M, many ? 64 : 8)), block(32, 8);
#define INPUTS(NC, RB) VN_LAUNCH_NAMED(ctx, "delta_inputs_kernel", (delta_inputs_kernel<T, NC, RB>), grid, block, 0, conv, in)
  if (many) { if (nc <= 1) INPUTS(1, 8); else if (nc <= 2) INPUTS(2, 8); else INPUTS(4, 8); return VN_OK; }
  if (nc <= 1) INPUTS(1, 1); else if (nc <= 2) INPUTS(2, 1); else if (nc <= 4) INPUTS(4, 1); else if (nc <= 8) INPUTS(8, 1); else INPUTS(16, 1);
#undef INPUTS
  return VN_OK;
}
template int32_t vn_delta_inputs<float>(vn_ctx*, const ConvIn<float>&, const DeltaIn&);
template int32_t vn_delta_inputs<__nv_bfloat16>(vn_ctx*, const ConvIn<__nv_bfloat16>&, const DeltaIn&);

template <typename T>
int32_t vn_delta_step(vn_ctx* ctx, const DeltaStepArgs<T>& a) {
  const dim3 grid(a.in.H, a.in.rows.M);
  const int d = a.in.d;
  const int extra = 3 * a.in.vd + a.in.ra_ld + a.in.rg_ld;
  VN_REQUIRE(ctx, extra + 24 * 32 <= 12000, "low-rank factors too wide for the step kernel");
#define STEP2(DK, NP) VN_LAUNCH_NAMED(ctx, "delta_step_kernel", (delta_step_kernel<T, DK, NP>), grid, DELTA_STEP_THREADS, \
                                      (size_t)(24 * DK + extra) * 4, a)
#define STEP(DK) do { if (a.in.vd <= 64) STEP2(DK, 1); else STEP2(DK, 2); } while (0)
  if (d <= 32) STEP(4); else if (d <= 64) STEP(8); else if (d <= 96) STEP(12); else if (d <= 128) STEP(16); else STEP2(32, 1);
#undef STEP2
#undef STEP
  return VN_OK;
}
template int32_t vn_delta_step<float>(vn_ctx*, const DeltaStepArgs<float>&);
template int32_t vn_delta_step<__nv_bfloat16>(vn_ctx*, const DeltaStepArgs<__nv_bfloat16>&);

int32_t vn_delta_scan(vn_ctx* ctx, const DeltaRuleArgs& a) {
  const int d = a.d;
  const bool vec = d % 4 == 0 && a.vd % 4 == 0;
  // more columns per group: fewer reads per column; fewer: more warps.  The widest that leaves two warps per scheduler
  const long long cols = (long long)a.rows.n_ent * a.H * a.vd;
  const int nc = d > 128 ? 4 : cols >= 16 * 8 * ctx->sm_count ? 8 : cols >= 16 * 4 * ctx->sm_count ? 4 : 2;
#define SCAN2(RPL, NC, VEC, W) do { const dim3 grid(ceil_div(a.vd, 2 * NC * W), a.H, a.rows.n_ent); \
    VN_LAUNCH_NAMED(ctx, "delta_scan_kernel", (delta_scan_kernel<RPL, NC, VEC, W>), grid, 32 * W, 0, a); } while (0)
#define SCAN(RPL, NC, W) do { if (vec) SCAN2(RPL, NC, 4, W); else SCAN2(RPL, NC, 1, W); } while (0)
  if (d <= 64) { if (nc == 8) SCAN(4, 8, 4); else if (nc == 4) SCAN(4, 4, 2); else SCAN(4, 2, 2); }
  else if (d <= 128) { if (nc == 8) SCAN(8, 8, 4); else if (nc == 4) SCAN(8, 4, 2); else SCAN(8, 2, 2); }
  else SCAN(16, 4, 2);
#undef SCAN
#undef SCAN2
  return VN_OK;
}
