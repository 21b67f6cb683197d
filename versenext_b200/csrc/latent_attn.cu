// Launches of the latent attention kernels.
#include "latent_attn.cuh"

namespace {

template <int NT, int MT>
int32_t launch_mma(vn_ctx* ctx, const LatentArgs& a) {
  const size_t smem = latent_detail::smem_bytes(MT, 32 * NT);
  static unsigned long long attr_set = 0;   // one bit per device
  if (!((attr_set >> (ctx->device & 63)) & 1ull)) {
    VN_CUDA(ctx, cudaFuncSetAttribute((latent_attn_mma_kernel<NT, MT>), cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    attr_set |= 1ull << (ctx->device & 63);
  }
  const dim3 grid(a.splits, ceil_div(a.rows.max_n * a.H, 16 * MT), a.rows.n_ent);
  VN_LAUNCH_NAMED(ctx, "latent_attn_mma_kernel", (latent_attn_mma_kernel<NT, MT>), grid, 128, smem, a);
  return VN_OK;
}

template <int NT>
int32_t launch_rows(vn_ctx* ctx, const LatentArgs& a) {
  const int t = latent_tile_rows(a.Rp, a.rows.max_n * a.H);
  if (t == 16) return launch_mma<NT, 1>(ctx, a);
  if (t == 32 || NT > 8) return launch_mma<NT, 2>(ctx, a);
  return launch_mma<NT, (NT > 8 ? 2 : 4)>(ctx, a);
}

template <typename T>
int32_t launch_simt(vn_ctx* ctx, const LatentArgs& a) {
  const dim3 grid(ceil_div(a.H, 8), a.rows.M);
  const int nr = a.Rp / 32;
#define LA(NR) VN_LAUNCH_NAMED(ctx, "latent_attn_kernel", (latent_attn_kernel<T, NR>), grid, 256, 0, a)
  if (nr <= 2) LA(2); else if (nr <= 4) LA(4); else if (nr <= 8) LA(8); else if (nr <= 16) LA(16); else LA(32);
#undef LA
  return VN_OK;
}

}  // namespace

int32_t vn_latent_attention(vn_ctx* ctx, const LatentArgs& a, bool bf16, bool mma) {
  if (!bf16) return launch_simt<float>(ctx, a);
  if (!mma) return launch_simt<__nv_bfloat16>(ctx, a);
  int32_t st;
  switch (a.Rp / 32) {
    case 1: st = launch_rows<1>(ctx, a); break;
    case 2: st = launch_rows<2>(ctx, a); break;
    case 3: st = launch_rows<3>(ctx, a); break;
    case 4: st = launch_rows<4>(ctx, a); break;
    case 6: st = launch_rows<6>(ctx, a); break;
    case 8: st = launch_rows<8>(ctx, a); break;
    case 10: st = launch_rows<10>(ctx, a); break;
    case 12: st = launch_rows<12>(ctx, a); break;
    case 16: st = launch_rows<16>(ctx, a); break;
    case 18: st = launch_rows<18>(ctx, a); break;
    default: return vn_fail(ctx, VN_ERR_UNSUPPORTED, "latent pitch %d", a.Rp);
  }
  if (st != VN_OK || a.splits <= 1) return st;
  VN_LAUNCH(ctx, latent_merge_kernel<__nv_bfloat16>, a.rows.M * a.H, 128, 0, a);
  return VN_OK;
}
