// Composed models: a list of layers of different kinds (latent attention, grouped-query attention, selective scan, state-space
// duality, gated delta rule, lightning attention), each with an optional feed-forward or mixture of experts and an optional
// input of its own for every token, and optionally a block of layers that is run several times with the same weights.  The
// residual is one stream that sublayers add to, or an arrangement of several (streams.cuh).
// Weights, the per-sequence cache (paged latents, keys and values, rings of convolution inputs and of recurrent states), and
// the forward over new rows of a uniform or a ragged batch.  Included by model.cu: it uses that file's GEMM helpers.
//
// One forward serves prompts, portions of prompts, single tokens and mixtures.  Projections of at most 256 rows of a
// bf16 model are split-K tcgen05 GEMMs whose slices are summed by the kernel that needs them; longer ones go through
// the tcgen05 segment kernel; an fp32 model uses the fp32 GEMM.  When every entry brings one token, a mixer's
// recurrence or attention and what surrounds it is one kernel (mamba_step_kernel, ssd_step_kernel, delta_step_kernel,
// attn_step_kernel, lightning_scan_kernel).
#pragma once
#include "json_value.h"
#include "latent_attn.cuh"
#include "lightning.cuh"
#include "paged_attn.cuh"
#include "router.cuh"
#include "scan_delta.cuh"
#include "scan_mamba.cuh"
#include "seq_ops.cuh"
#include "ssd.cuh"
#include "streams.cuh"

namespace hybrid {

enum Kind { LATENT = 0, MAMBA1 = 1, DELTA = 2, ATTENTION = 3, LIGHTNING = 4, MAMBA2 = 5 };
enum Gate { GATE_NONE = 0, GATE_HEAD = 1, GATE_ELEMENT = 2 };       // output gates of attention layers

struct HLayer {
  int kind = 0;
  // latent: H, d, vd, R (kv_rank), window, scale.  mamba: inner, dt_rank, nstate, taps.  delta: H, KH, d, vd, taps, ra, rg
  int H = 0, KH = 0, d = 0, vd = 0, R = 0, window = 0, taps = 1, inner = 0, dt_rank = 0, nstate = 0, ra = 0, rg = 0;
  float scale = 1.f;
  // attention: H, KH, d, vd, taps, window, scale and the line below (conv_named: the convolutions are in the checkpoint).
  // lightning: H, d, vd, decay
  int kv_from = -1, gated = GATE_NONE, P = 0, rd = 0, rope = -1, conv_named = 0;
  int chunk = 0, qk_norm = 0, bias = 0, out_bias = 0, temps = 0, interleaved = 0;
  float softcap = 0.f;
  // latent, besides: rotated dimensions rr, what the output gate multiplies, sink.  mamba2: H, vd, nstate, taps, groups, norm_groups
  int rr = 0, gate = GATE_HEAD, sinks = 1, groups = 1, norm_groups = 1;
  std::vector<double> decay;
  int ff = 0, act = GLU_SILU;      // feed-forward width (0: none), function of its gate and up
  float limit = 0.f;               // of GLU_CLAMP
  // mixture: n_exp experts of width ff and n_id identity experts (0: a dense feed-forward), of which a row uses `top`, out of
  // the `keep` best of exp_groups groups
  int n_exp = 0, n_id = 0, top = 0, exp_groups = 1, keep = 1, corrected = 0;
  int sigmoid = 0, weigh_input = 0;    // scores by sigmoid; a weight multiplies the expert's input instead of its result
  int sff = 0, sffp = 0;           // width of the gated expert that serves every row (0: none)
  float s_limit = 0.f;
  int ff_plain = 0;                // no gate: squared relu
  int poly = 0;                    // no gate: PolyNorm
  int dp = 0, Rp = 0, dtp = 0, rap = 0, rgp = 0, n_in = 0, n_x = 0, ffp = 0;    // padded sizes
  float* norm1 = nullptr; float* norm2 = nullptr;                               // 1 + stored weight
  float* post[2] = {nullptr, nullptr};                                          // norms of the sublayers' results
  void* w_in = nullptr;            // first projection, all its parts stacked [n_in, D]
  void* w_o = nullptr;
  void* w_uk = nullptr;            // latent: per head W_uk^T [H][Rp][dp];  delta: a2 [H d, rap];  mamba: dt [inner, dtp]
  void* w_uv = nullptr;            // latent: [H][vd][Rp];                  delta: g2 [H vd, rgp];  mamba: x [n_x, inner]
  float* f_a = nullptr;            // latent: norm of the latent;  delta: norm [vd];       mamba: A = -exp(A_log);  lightning: norm [H vd]
  float* f_b = nullptr;            // latent: sink [H];            delta: exp(A_log) [H];  mamba: D;                lightning: decay [H][2]
  float* f_c = nullptr;            //                              delta: dt_bias [H d];   mamba: dt bias;          lightning: powers [H][65]
  // residual arrangement, per sublayer (0 mixer, 1 feed-forward)
  float *hc_in[2] = {nullptr, nullptr}, *hc_out[2] = {nullptr, nullptr}, *hc_mix[2] = {nullptr, nullptr};
  void* w_rg[2] = {nullptr, nullptr};     // gate of the sublayer's result; of a plain feed-forward: the rows behind w_gu's
  float* rg_b[2] = {nullptr, nullptr};
  float* in_conv = nullptr;               // [D, taps] convolution of what the mixer reads
  float* conv = nullptr; float* conv_b = nullptr;
  void* w_gu = nullptr; void* w_down = nullptr;                                 // of a mixture: per expert
  float* f_d = nullptr;                   // mamba2: -exp(A_log) [H]
  float* o_b = nullptr;                   // bias of the output projection
  float* temp = nullptr;                  // attention: factors of the heads' scores [H]
  float* coef = nullptr;                  // PolyNorm's four numbers
  void *w_sgu = nullptr, *w_sdown = nullptr;                                    // of the expert that serves every row
  void* w_router = nullptr; float* correction = nullptr;                        // [n_router, D], [n_out]
  void *w_sgate = nullptr, *w_sproj = nullptr; float* s_norm = nullptr;         // the token's own input
  int n_out() const { return n_exp + n_id; }
  int n_router() const { return sff ? (n_out() + 8) & ~7 : n_out(); }          // the shared expert's gate is row n_out
  // the shared expert is stored, and run, as one more of the others where it has their shape
  int joined() const { return sff == ff && sff && s_limit == limit && !n_id && top < MAX_CHOSEN; }
  int n_mats() const { return n_exp + joined(); }
  int slots() const { return top + joined(); }
  int single_up() const { return ff_plain || poly; }                            // one matrix in front of the activation
  int attn_gates() const { return gated == GATE_HEAD ? H : gated ? H * vd : 0; }
  int n_gate() const { return gate == GATE_HEAD ? H : gate == GATE_ELEMENT ? H * vd : 0; }      // latent
  int conv_ch() const {
    if (kind == MAMBA1) return inner;
    if (kind == MAMBA2) return inner + 2 * groups * nstate;
    if (kind == ATTENTION) return H * d + (kv_from < 0 ? KH * (d + vd) : 0);
    return 2 * KH * d + H * vd;
  }
  long long state_elems() const { return kind == MAMBA1 || kind == MAMBA2 ? (long long)inner * nstate : (long long)H * d * vd; }
};

struct Run { int layer; int pass; int kv_run; };      // pass: -1 outside the loop; kv_run: the run whose keys it reads

struct Rope {                      // frequencies of the rotated pairs, amplitude of cos and sin
  std::vector<double> freq;
  float amp = 1.f;
  float2* table = nullptr;         // [rows][pairs]
  int rows = 0;
};

struct Model {
  int D = 0, vocab = 0, sinusoidal = 0;
  float eps = 1e-6f;
  std::vector<HLayer> layers;
  int loop_start = 0, loop_stop = 0, loop_times = 0;
  bool loop_add = false;           // a pass begins with x + x0 (but the first) + step vector, else with W [x | x0] + step vector
  bool post_norm = false;          // norms of the sublayers' results
  bool tied = false;               // the head is the embedding table
  std::vector<Run> runs;
  void* w_loop = nullptr;          // [D, 2 D]
  float* loop_step = nullptr;      // [times, D]
  double* freq = nullptr;          // [ceil(D / 2)]
  std::set<std::string> want;
  float* x0 = nullptr; void* cat = nullptr; char* ws = nullptr; size_t ws_bytes = 0;
  int* meta = nullptr; int meta_cap = 0;
  float* probe = nullptr;          // residual stream after every layer run, [runs][M][D], or null
  // arrangement of the residual
  int layer_norm = 0, streams = 0, in_taps = 0, res_gate = 0;     // streams 0: one stream that sublayers add to
  bool arranged = false;           // the forward goes through streams.cuh
  bool plain_norm = false;         // norm weights are stored as they are, not around zero
  int side = 0, sidep = 0;         // width of the tokens' own inputs per layer (0: none), padded
  void* side_embed = nullptr;      // [V, layers * side]
  int *exp_count = nullptr, *exp_cur = nullptr, *exp_off = nullptr;    // per expert: rows (zero between forwards), fill level, first row
  int max_out = 0;
  std::vector<Rope> ropes;
  std::vector<void*> retired;      // tables replaced by longer ones (a captured graph may still read them)
  void* hc = nullptr;              // [rows, D] what the mixer reads
  float *gate = nullptr, *y = nullptr;                            // [rows, D] raw gates; result of a sublayer
  float* gate_ws = nullptr; size_t gate_ws_bytes = 0;             // split-K slices of a gate
  float* seg = nullptr; size_t seg_bytes = 0;                     // LightningArgs::seg_state, SsdArgs::seg_state and seg_decay
};

// what a cache of such a model keeps besides the lengths; owned by the root cache, shared by its views
struct Cache {
  int pending = 1, ring_len = 2;   // rows that can be appended and cut back; state snapshots per sequence
  bool pooled = false;
  int max_pages = 0, n_pages = 0, slots = 0;
  int* table_dev = nullptr;
  std::vector<int> table, used;    // [slots][max_pages]; pages held by each slot
  std::vector<int> free_pages;
  std::vector<void*> ring, in_ring;   // per layer run: inputs of the mixer's convolutions (attention), of the input convolution
};

inline int up8(int n) { return (n + 7) & ~7; }
inline int up4(int n) { return (n + 3) & ~3; }
// latent rows are padded to a multiple of 32 that the tensor-core kernel has an instance for
inline int latent_pitch(int R) {
  static const int tiles[] = {1, 2, 3, 4, 6, 8, 10, 12, 16, 18};
  for (int t : tiles)
    if (R <= 32 * t) return 32 * t;
  return (R + 31) & ~31;
}

struct Arena {
  char* base = nullptr;
  size_t off = 0;
  template <typename P> void take(P** p, size_t bytes) {
    *p = base ? reinterpret_cast<P*>(base + off) : nullptr;
    off += (bytes + 255) & ~size_t(255);
  }
};
struct Buffers {
  float* proj = nullptr;           // [M, n_in] when the projection is not split (also [M, D] of the loop entry)
  void* mix = nullptr;             // [M, H vd | inner] input of the output projection
  void* act = nullptr;             // [M, ffp]
  void *q = nullptr, *qc = nullptr, *oc = nullptr;                    // latent
  float *gate = nullptr, *part_o = nullptr, *part_ml = nullptr;
  void *xc = nullptr, *z = nullptr, *dtb = nullptr; float *p = nullptr, *dt = nullptr;       // mamba
  float *dq = nullptr, *dk = nullptr, *dv = nullptr, *beta = nullptr, *g = nullptr, *gg = nullptr, *o = nullptr;   // delta
  void *low_a = nullptr, *low_g = nullptr;
  void* lin = nullptr; float* ss = nullptr;      // lightning
  void* gate_t = nullptr;                        // latent: output gates in the storage dtype
  void *xbc = nullptr, *u = nullptr;             // mamba2
  // mixture of experts
  float *logits = nullptr, *slot_w = nullptr, *sorted_w = nullptr, *sgate = nullptr, *sy = nullptr;
  void* sact = nullptr;
  int *slot_expert = nullptr, *slot_pos = nullptr, *sorted_row = nullptr, *sub_seg = nullptr;
  void *hs = nullptr, *ey = nullptr;
  int sub_cap = 0;
  void* side_act = nullptr;
};
constexpr int SPLIT_ROWS = 64, MAX_SPLITS = 16;   // key splits of the latent attention: forwards of few rows

inline void layout(const Model& hm, const HLayer& L, size_t M, size_t e, Arena& A, Buffers& b) {
  A.off = 0;
  A.take(&b.proj, M * std::max(std::max(L.n_in, hm.D), L.single_up() ? L.ffp + hm.D : 0) * 4);
  A.take(&b.mix, M * (size_t)(L.kind == MAMBA1 ? L.inner : L.H * L.vd) * e);
  if (L.ff) A.take(&b.act, M * std::max(1, L.slots()) * L.ffp * e);
  if (L.n_exp) {
    const size_t slots = M * L.slots();
    A.take(&b.logits, M * L.n_router() * 4);
    A.take(&b.slot_w, slots * 4);
    A.take(&b.slot_expert, slots * 4);
    A.take(&b.slot_pos, slots * 4);
    A.take(&b.sorted_row, slots * 4);
    A.take(&b.sorted_w, slots * 4);
    if (L.sff) A.take(&b.sgate, M * 4);
    if (L.sff && !L.joined()) {
      A.take(&b.sact, M * L.sffp * e);
      A.take(&b.sy, M * hm.D * 4);
    }
    A.take(&b.hs, slots * hm.D * e);
    A.take(&b.ey, slots * hm.D * e);
    b.sub_cap = (int)(L.n_mats() + slots / 256 + 1);
    A.take(&b.sub_seg, (size_t)3 * b.sub_cap * 4);
  }
  if (hm.side) A.take(&b.side_act, M * hm.sidep * e);
  if (L.kind == LATENT) {
    A.take(&b.q, M * L.H * L.dp * e);
    A.take(&b.qc, M * L.H * L.Rp * e);
    A.take(&b.oc, M * L.H * L.Rp * e);
    if (L.gate == GATE_HEAD) A.take(&b.gate, M * L.H * 4);
    if (L.gate == GATE_ELEMENT) A.take(&b.gate_t, M * L.H * L.vd * e);
    if (M <= SPLIT_ROWS) {
      A.take(&b.part_o, (size_t)MAX_SPLITS * M * L.H * L.Rp * 4);
      A.take(&b.part_ml, (size_t)MAX_SPLITS * M * L.H * 2 * 4);
    }
  } else if (L.kind == MAMBA1) {
    A.take(&b.xc, M * L.inner * e);
    A.take(&b.z, M * L.inner * e);
    A.take(&b.dtb, M * L.dtp * e);
    A.take(&b.p, M * L.n_x * 4);
    A.take(&b.dt, M * L.inner * 4);
  } else if (L.kind == MAMBA2) {
    A.take(&b.xbc, M * up8(L.conv_ch()) * e);
    A.take(&b.dt, M * L.H * 4);
    A.take(&b.u, M * L.inner * e);
    A.take(&b.z, M * L.inner * e);
  } else if (L.kind == ATTENTION) {
    A.take(&b.q, M * L.H * L.P * e);
    if (M <= SPLIT_ROWS) {
      A.take(&b.part_o, (size_t)MAX_SPLITS * M * L.H * L.P * 4);
      A.take(&b.part_ml, (size_t)MAX_SPLITS * M * L.H * 2 * 4);
    }
  } else if (L.kind == LIGHTNING) {
    A.take(&b.lin, M * L.n_in * e);
    A.take(&b.ss, M * L.H * ceil_div(L.vd, 64) * 4 * 4);
  } else {
    A.take(&b.dq, M * L.KH * L.d * 4);
    A.take(&b.dk, M * L.KH * L.d * 4);
    A.take(&b.dv, M * L.H * L.vd * 4);
    A.take(&b.beta, M * L.H * 4);
    A.take(&b.g, M * L.H * L.d * 4);
    A.take(&b.gg, M * L.H * L.vd * 4);
    A.take(&b.o, M * L.H * L.vd * 4);
    A.take(&b.low_a, M * L.rap * e);
    A.take(&b.low_g, M * L.rgp * e);
  }
}

// Rotary frequencies f_i = base^(-2 i / dims).  Linear scaling divides them all by `factor`; scaling by wavelength divides those
// with fewer than `low` turns over the original context, keeps those with more than `high`, and blends linearly in the number of
// turns between the two (Llama 3.1); YaRN does it with a ramp over the pairs.
inline Rope make_rope(const JsonValue& r) {
  Rope out;
  const int dims = (int)r.number("dims", 0);
  const double base = r.number("base", 10000.0);
  for (int i = 0; i < dims / 2; ++i) out.freq.push_back(pow(base, -2.0 * i / dims));
  const JsonValue* s = r.find("scaling");
  if (!s || s->kind != JsonValue::OBJ) return out;
  const double factor = s->number("factor", 1), original = s->number("original", 1);
  if (s->text("kind") == "linear") {
    for (double& f : out.freq) f /= factor;
    return out;
  }
  if (s->text("kind") == "wavelength") {
    const double low = s->number("low", 1), high = s->number("high", 4);
    for (double& f : out.freq) {
      const double wave = 2 * M_PI / f;
      if (wave < original / high) continue;
      const double share = wave > original / low ? 0.0 : (original / wave - low) / (high - low);
      f = (1 - share) * f / factor + share * f;
    }
    return out;
  }
  auto dim_of = [&](double turns) { return dims * log(original / (2 * M_PI * turns)) / (2 * log(base)); };
  const double lo = std::max(floor(dim_of(s->number("fast", 32))), 0.0);
  const double hi = std::min(ceil(dim_of(s->number("slow", 1))), dims - 1.0);
  for (int i = 0; i < dims / 2; ++i) {
    const double ramp = std::min(std::max((i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
    out.freq[i] = out.freq[i] / factor * ramp + out.freq[i] * (1 - ramp);
  }
  out.amp = (float)(0.1 * log(factor) + 1.0);
  return out;
}

// ---- configuration ---------------------------------------------------------------------------------------------
int32_t parse(vn_ctx* ctx, const JsonValue& j, Model* hm, Config* c) {
  c->vocab = (int)j.number("vocab_size", 0);
  c->dim = (int)j.number("dim", 0);
  const std::string dt = j.text("dtype");
  VN_REQUIRE(ctx, dt.empty() || dt == "f32" || dt == "bf16", "dtype must be \"f32\" or \"bf16\", got %s", dt.c_str());
  c->bf16 = dt == "bf16";
  c->tie = hm->tied = j.number("tie_weights", 0) != 0;
  c->max_seq_len = (int)j.number("max_seq_len", 2048);
  hm->D = c->dim; hm->vocab = c->vocab;
  hm->eps = (float)j.number("norm_eps", 1e-6);
  hm->sinusoidal = j.text("positions") == "sinusoidal";
  const std::string norm = j.text("norm");
  VN_REQUIRE(ctx, norm.empty() || norm == "rms" || norm == "layer", "norm %s unknown (rms | layer)", norm.c_str());
  hm->layer_norm = norm == "layer";
  hm->streams = (int)j.number("streams", 0);
  hm->in_taps = (int)j.number("input_conv", 0);
  hm->res_gate = j.number("residual_gate", 0) != 0;
  VN_REQUIRE(ctx, hm->streams >= 0 && hm->streams <= MAX_STREAMS && hm->in_taps >= 0, "streams (at most %d) or input_conv out of range", MAX_STREAMS);
  hm->arranged = hm->layer_norm || hm->streams || hm->in_taps || hm->res_gate;
  const std::string nw = j.text("norm_weight");
  VN_REQUIRE(ctx, nw.empty() || nw == "plain" || nw == "around_zero", "norm_weight %s unknown (plain | around_zero)", nw.c_str());
  hm->plain_norm = hm->layer_norm || nw == "plain";
  hm->post_norm = j.number("post_norm", 0) != 0;
  hm->side = (int)j.number("token_side", 0);
  hm->sidep = up8(hm->side);
  VN_REQUIRE(ctx, hm->side >= 0, "token_side out of range");
  const JsonValue* ls = j.find("layers");
  VN_REQUIRE(ctx, c->vocab > 0 && c->dim > 0 && ls && ls->kind == JsonValue::ARR && !ls->arr.empty(),
             "a composed model needs vocab_size, dim and layers");
  for (size_t i = 0; i < ls->arr.size(); ++i) {
    const JsonValue& l = ls->arr[i];
    HLayer L;
    const std::string t = l.text("mixer");
    auto I = [&](const char* k, int dflt = 0) { return (int)l.number(k, dflt); };
    L.kind = t == "latent_attention" ? LATENT : t == "mamba1" ? MAMBA1 : t == "channel_delta" ? DELTA : t == "attention" ? ATTENTION
             : t == "lightning" ? LIGHTNING : t == "mamba2" ? MAMBA2 : -1;
    VN_REQUIRE(ctx, L.kind >= 0, "layer %zu: mixer %s unknown (latent_attention | attention | mamba1 | mamba2 | channel_delta | lightning)", i, t.c_str());
    auto rope = [&](int dims) -> int32_t {       // the layer's rotation, at most `dims` dimensions
      const JsonValue* r = l.find("rope");
      if (!r || r->kind != JsonValue::OBJ) return VN_OK;
      const Rope made = make_rope(*r);
      L.rd = 2 * (int)made.freq.size();
      VN_REQUIRE(ctx, L.rd <= dims, "layer %zu: %d of %d dimensions rotated", i, L.rd, dims);
      for (size_t k = 0; k < hm->ropes.size() && L.rope < 0; ++k)
        if (hm->ropes[k].freq == made.freq && hm->ropes[k].amp == made.amp) L.rope = (int)k;
      if (L.rope < 0) { L.rope = (int)hm->ropes.size(); hm->ropes.push_back(made); }
      L.interleaved = r->number("interleaved", 0) != 0;
      return VN_OK;
    };
    L.ff = I("mlp_hidden");
    const std::string act = l.text("mlp_act");
    VN_REQUIRE(ctx, !L.ff || act == "gelu_tanh" || act == "silu" || act == "clamped" || act == "relu2" || act == "poly_norm",
               "layer %zu: activation %s unknown (gelu_tanh | silu | clamped | relu2 | poly_norm)", i, act.c_str());
    L.act = act == "gelu_tanh" ? GLU_GELU : act == "clamped" ? GLU_CLAMP : GLU_SILU;
    L.limit = (float)l.number("mlp_limit", 0);
    L.ff_plain = act == "relu2";
    L.poly = act == "poly_norm";
    if (const JsonValue* x = l.find("experts"))
      if (x->kind == JsonValue::OBJ) {
        L.n_exp = (int)x->number("count", 0); L.n_id = (int)x->number("identity", 0); L.top = (int)x->number("top", 0);
        L.exp_groups = (int)x->number("groups", 1); L.keep = (int)x->number("keep", L.exp_groups);
        L.corrected = x->number("correction", 0) != 0;
        const std::string score = x->text("score"), weight = x->text("weight");
        VN_REQUIRE(ctx, (score.empty() || score == "softmax" || score == "sigmoid") && (weight.empty() || weight == "result" || weight == "input"),
                   "layer %zu: experts' score %s (softmax | sigmoid) or weight %s (result | input) unknown", i, score.c_str(), weight.c_str());
        L.sigmoid = score == "sigmoid";
        L.weigh_input = weight == "input";
        if (const JsonValue* sh = x->find("shared"))
          if (sh->kind == JsonValue::OBJ) {
            L.sff = (int)sh->number("hidden", 0);
            L.s_limit = (float)sh->number("limit", L.limit);
            L.sffp = up8(L.sff);
            VN_REQUIRE(ctx, L.sff > 0, "layer %zu: shared expert of width %d", i, L.sff);
          }
        VN_REQUIRE(ctx, !(L.weigh_input && L.n_id), "layer %zu: identity experts take their weights on the result", i);
        const int n = L.n_out();
        VN_REQUIRE(ctx, L.ff > 0 && !L.single_up() && L.n_exp > 0 && L.n_id >= 0 && n <= 1024 && L.exp_groups >= 1 && n % L.exp_groups == 0 &&
                   L.keep >= 1 && L.keep <= L.exp_groups && L.top >= 1 && L.top <= MAX_CHOSEN && L.top <= L.keep * (n / L.exp_groups),
                   "layer %zu: mixture of %d experts and %d identities in %d groups, %d kept, %d chosen", i, L.n_exp, L.n_id, L.exp_groups, L.keep, L.top);
        hm->max_out = std::max(hm->max_out, n + L.joined());
      }
    if (L.ff_plain || L.kind == LIGHTNING) hm->arranged = true;
    L.ffp = up8(L.ff);
    L.H = I("heads"); L.d = I("dim"); L.vd = I("vdim"); L.taps = I("conv", 1);
    if (L.kind == LATENT) {
      L.R = I("kv_rank"); L.window = I("window"); L.scale = (float)l.number("scale", 0);
      L.rr = I("rot_dim"); L.sinks = l.number("sink", 1) != 0;
      const std::string gate = l.text("output_gate");
      VN_REQUIRE(ctx, gate.empty() || gate == "head" || gate == "element" || gate == "none", "layer %zu: output gate %s unknown (head | element | none)", i, gate.c_str());
      L.gate = gate == "none" ? GATE_NONE : gate == "element" ? GATE_ELEMENT : GATE_HEAD;
      VN_REQUIRE(ctx, L.H > 0 && L.d > 0 && L.vd > 0 && L.R > 0 && L.rr >= 0 && L.rr % 2 == 0 && L.R + L.rr <= 1024 && L.window >= 0, "layer %zu: latent attention sizes", i);
      TRY(rope(L.rr));
      VN_REQUIRE(ctx, L.rd == L.rr && (!L.rr || L.interleaved), "layer %zu: the rotated part of %d dimensions needs a rotation of as many interleaved ones", i, L.rr);
      L.dp = up8(L.d); L.Rp = latent_pitch(L.R + L.rr);
      L.n_in = up8(L.H * (L.d + L.rr) + L.R + L.rr + L.n_gate());
    } else if (L.kind == MAMBA1) {
      L.inner = I("inner"); L.dt_rank = I("dt_rank"); L.nstate = I("state");
      VN_REQUIRE(ctx, L.inner > 0 && L.dt_rank > 0 && L.nstate > 0 && L.nstate <= 128 && L.taps >= 1, "layer %zu: selective scan sizes", i);
      L.dtp = up8(L.dt_rank);
      L.n_in = 2 * L.inner;
      L.n_x = up8(L.dtp + 2 * L.nstate);
    } else if (L.kind == MAMBA2) {
      L.inner = L.H * L.vd; L.nstate = I("state"); L.groups = I("groups", 1); L.norm_groups = I("norm_groups", 1);
      VN_REQUIRE(ctx, L.H > 0 && L.vd > 0 && L.nstate > 0 && L.nstate <= 512 && L.groups > 0 && L.H % L.groups == 0 && L.norm_groups > 0 &&
                 L.inner % L.norm_groups == 0 && L.taps >= 1, "layer %zu: state-space sizes", i);
      L.n_in = up8(2 * L.inner + 2 * L.groups * L.nstate + L.H);
    } else if (L.kind == ATTENTION) {
      L.KH = I("kv_heads"); L.window = I("window"); L.scale = (float)l.number("scale", 0); L.kv_from = I("kv_from", -1);
      L.chunk = I("chunk"); L.softcap = (float)l.number("softcap", 0); L.qk_norm = l.number("qk_norm", 0) != 0; L.bias = l.number("bias", 0) != 0;
      const std::string gate = l.text("output_gate");
      VN_REQUIRE(ctx, gate.empty() || gate == "head" || gate == "element" || gate == "none", "layer %zu: output gate %s unknown (head | element | none)", i, gate.c_str());
      L.gated = gate == "head" ? GATE_HEAD : gate == "element" || (gate.empty() && l.number("output_gate", 0) != 0) ? GATE_ELEMENT : GATE_NONE;
      L.out_bias = l.number("out_bias", L.bias) != 0;
      L.temps = l.number("temperature", 0) != 0;
      L.conv_named = l.find("conv") && l.find("conv")->kind == JsonValue::NUM;
      TRY(rope(L.d));
      VN_REQUIRE(ctx, !(L.conv_named && (L.qk_norm || L.bias)) && !(L.kv_from >= 0 && L.qk_norm), "layer %zu: norms and biases of the heads together with "
                 "convolutions, or norms of another layer's keys", i);
      VN_REQUIRE(ctx, L.chunk >= 0 && L.softcap >= 0.f && L.H > 0 && L.KH > 0 && L.H % L.KH == 0 && L.d > 0 && L.vd > 0 && L.d <= 1024 && L.vd <= 1024 && L.rd <= L.d &&
                 L.window >= 0 && L.taps >= 1, "layer %zu: attention sizes", i);
      if (L.kv_from >= 0) {
        VN_REQUIRE(ctx, L.kv_from < (int)i, "layer %zu: keys and values of layer %d, which does not run before it", i, L.kv_from);
        const HLayer& src = hm->layers[L.kv_from];
        VN_REQUIRE(ctx, src.kind == ATTENTION && src.kv_from < 0 && src.KH == L.KH && src.d == L.d && src.vd == L.vd,
                   "layer %zu: keys and values of layer %d have other sizes, or are not its own", i, L.kv_from);
      }
      L.P = attn_pitch(std::max(L.d, L.vd));
      L.n_in = up8(L.conv_ch() + L.attn_gates());
    } else if (L.kind == LIGHTNING) {
      const JsonValue* dec = l.find("decay");
      VN_REQUIRE(ctx, L.H > 0 && L.d > 0 && L.d <= 512 && L.vd > 0 && dec && dec->kind == JsonValue::ARR && (int)dec->arr.size() == L.H,
                 "layer %zu: lightning attention sizes, or not one decay per head", i);
      for (auto& v : dec->arr) L.decay.push_back(v.num);
      L.n_in = up8(2 * L.H * (L.d + L.vd));
    } else {
      L.KH = I("kv_heads"); L.ra = I("decay_rank"); L.rg = I("gate_rank");
      VN_REQUIRE(ctx, L.H > 0 && L.KH > 0 && L.H % L.KH == 0 && L.d > 0 && L.d <= 256 && L.vd > 0 && L.vd <= 512 && L.ra > 0 &&
                 L.rg > 0 && L.taps >= 1, "layer %zu: delta rule sizes", i);
      L.rap = up8(L.ra); L.rgp = up8(L.rg);
      L.n_in = up8(2 * L.KH * L.d + L.H * L.vd + L.H + L.ra + L.rg);
    }
    hm->layers.push_back(L);
  }
  const int n = (int)hm->layers.size();
  if (const JsonValue* lp = j.find("loop")) {
    if (lp->kind == JsonValue::OBJ) {
      hm->loop_start = (int)lp->number("start", 0);
      hm->loop_stop = (int)lp->number("stop", 0);
      hm->loop_times = (int)lp->number("times", 0);
      VN_REQUIRE(ctx, hm->loop_start >= 0 && hm->loop_start < hm->loop_stop && hm->loop_stop <= n && hm->loop_times >= 1,
                 "loop over layers %d .. %d, %d times, of %d layers", hm->loop_start, hm->loop_stop, hm->loop_times, n);
      const std::string entry = lp->text("entry");
      VN_REQUIRE(ctx, entry.empty() || entry == "project" || entry == "add", "entry of a looped block %s unknown (project | add)", entry.c_str());
      hm->loop_add = entry == "add";
    }
  }
  const int a = hm->loop_times ? hm->loop_start : n, b = hm->loop_times ? hm->loop_stop : n;
  std::vector<int> last(n, -1);           // latest run of a layer
  auto run = [&](int i, int t) {
    const int from = hm->layers[i].kv_from;
    last[i] = (int)hm->runs.size();
    hm->runs.push_back({i, t, from < 0 ? last[i] : last[from]});
  };
  for (int i = 0; i < a; ++i) run(i, -1);
  for (int t = 0; t < hm->loop_times; ++t)
    for (int i = a; i < b; ++i) run(i, t);
  for (int i = b; i < n; ++i) run(i, -1);
  VN_REQUIRE(ctx, !hm->arranged || !hm->loop_times, "a looped block needs the plain residual");
  VN_REQUIRE(ctx, !hm->side || !hm->loop_times, "tokens' own inputs do not go with a looped block");
  if (hm->arranged)
    for (const HLayer& L : hm->layers)
      VN_REQUIRE(ctx, !L.n_exp && !hm->side && L.kind != MAMBA2 && !L.bias && !L.out_bias && !L.poly && !hm->post_norm,
                 "mixtures, state-space layers, biases, PolyNorm, norms of results and tokens' own inputs need the plain residual");
  return VN_OK;
}

int32_t zalloc(vn_model* m, void** p, size_t bytes) {
  TRY(dev_alloc(m->ctx, p, bytes));
  m->param_bytes += bytes;
  VN_CUDA(m->ctx, cudaMemsetAsync(*p, 0, bytes ? bytes : 16, m->ctx->stream));
  return VN_OK;
}

int32_t alloc(vn_model* m) {
  Model& hm = *m->hyb;
  const size_t e = m->esz, D = hm.D;
  auto W = [&](void** p, size_t n) { return zalloc(m, p, n * e); };
  auto F = [&](float** p, size_t n) { return zalloc(m, (void**)p, n * 4); };
  TRY(W(&m->emb, hm.vocab * D));
  if (hm.tied) m->head = m->emb; else TRY(W(&m->head, hm.vocab * D));
  TRY(F(&m->norm_f, D));
  TRY(dev_alloc(m->ctx, (void**)&m->status, 4));
  VN_CUDA(m->ctx, cudaMemsetAsync(m->status, 0, 4, m->ctx->stream));
  hm.want = {"embed", "final.norm"};
  if (!hm.tied) hm.want.insert("head");
  if (hm.loop_times) {
    TRY(F(&hm.loop_step, hm.loop_times * D));
    hm.want.insert("loop.step");
    if (!hm.loop_add) {
      TRY(W(&hm.w_loop, D * 2 * D));
      hm.want.insert("loop.in");
    }
  }
  if (hm.side) {
    TRY(W(&hm.side_embed, (size_t)hm.vocab * hm.layers.size() * hm.side));
    hm.want.insert("side.embed");
  }
  if (hm.max_out) {
    void* p[3] = {nullptr, nullptr, nullptr};
    for (void*& q : p) TRY(zalloc(m, &q, (size_t)hm.max_out * 4));
    hm.exp_count = (int*)p[0]; hm.exp_cur = (int*)p[1]; hm.exp_off = (int*)p[2];
  }
  if (hm.sinusoidal) {
    std::vector<double> f((D + 1) / 2);
    for (size_t i = 0; i < f.size(); ++i) f[i] = pow(10000.0, -2.0 * (double)i / (double)D);
    TRY(dev_alloc(m->ctx, (void**)&hm.freq, f.size() * 8));
    VN_CUDA(m->ctx, cudaMemcpyAsync(hm.freq, f.data(), f.size() * 8, cudaMemcpyHostToDevice, m->ctx->stream));
    VN_CUDA(m->ctx, cudaStreamSynchronize(m->ctx->stream));
  }
  for (size_t i = 0; i < hm.layers.size(); ++i) {
    HLayer& L = hm.layers[i];
    const std::string p = "l" + std::to_string(i) + ".";
    auto need = [&](std::initializer_list<const char*> names) { for (const char* s : names) hm.want.insert(p + s); };
    TRY(F(&L.norm1, D));
    TRY(W(&L.w_in, (size_t)L.n_in * D));
    need({"norm1", "mix.o"});
    if (L.kind == LATENT) {
      TRY(W(&L.w_uk, (size_t)L.H * L.Rp * L.dp));
      TRY(W(&L.w_uv, (size_t)L.H * L.vd * L.Rp));
      TRY(W(&L.w_o, D * L.H * L.vd));
      TRY(F(&L.f_a, L.R));
      TRY(F(&L.f_b, L.H));
      need({"mix.q", "mix.dkv", "mix.dkv.norm", "mix.uk", "mix.uv"});
      if (L.sinks) need({"mix.sink"});
      if (L.gate) need({"mix.g"});
    } else if (L.kind == ATTENTION) {
      TRY(W(&L.w_o, D * L.H * L.vd));
      TRY(F(&L.conv, (size_t)L.conv_ch() * L.taps));
      if (!L.conv_named) {                                 // one tap of weight 1: the projection itself
        const std::vector<float> unit(L.conv_ch(), 1.f);
        TRY(upload(m, unit.data(), L.conv, 1, L.conv_ch(), L.conv_ch(), 1, 0, true));
      }
      need({"mix.q"});
      if (L.kv_from < 0) need({"mix.k", "mix.v"});
      if (L.gated) need({"mix.g"});
      if (L.qk_norm) {
        TRY(F(&L.f_a, L.d));
        TRY(F(&L.f_b, L.d));
        need({"mix.q.norm", "mix.k.norm"});
      }
      if (L.bias) {
        TRY(F(&L.f_c, L.conv_ch()));
        need({"mix.q.b"});
        if (L.kv_from < 0) need({"mix.k.b", "mix.v.b"});
      }
      if (L.out_bias) { TRY(F(&L.o_b, D)); need({"mix.o.b"}); }
      if (L.temps) { TRY(F(&L.temp, L.H)); need({"mix.temp"}); }
      if (L.conv_named) need({"mix.q.conv"});
      if (L.conv_named && L.kv_from < 0) need({"mix.k.conv", "mix.v.conv"});
    } else if (L.kind == LIGHTNING) {
      TRY(W(&L.w_o, D * L.H * L.vd));
      TRY(F(&L.f_a, (size_t)L.H * L.vd));
      TRY(F(&L.f_b, (size_t)2 * L.H));
      TRY(F(&L.f_c, (size_t)65 * L.H));
      std::vector<float> dec, pw;
      for (double v : L.decay) {
        dec.push_back((float)v);
        dec.push_back((float)(v - (double)dec.back()));
        for (int k = 0; k <= 64; ++k) pw.push_back((float)pow(v, k));
      }
      TRY(upload(m, dec.data(), L.f_b, 1, (long long)dec.size(), (long long)dec.size(), 1, 0, true));
      TRY(upload(m, pw.data(), L.f_c, 1, (long long)pw.size(), (long long)pw.size(), 1, 0, true));
      need({"mix.q", "mix.k", "mix.v", "mix.g", "mix.norm"});
    } else if (L.kind == MAMBA2) {
      TRY(W(&L.w_o, D * L.inner));
      TRY(F(&L.f_a, L.inner));
      TRY(F(&L.f_b, L.H));
      TRY(F(&L.f_c, L.H));
      TRY(F(&L.f_d, L.H));
      TRY(F(&L.conv, (size_t)L.conv_ch() * L.taps));
      TRY(F(&L.conv_b, L.conv_ch()));
      need({"mix.in", "mix.conv", "mix.conv.b", "mix.dt_bias", "mix.A_log", "mix.D", "mix.norm"});
    } else if (L.kind == MAMBA1) {
      TRY(W(&L.w_uk, (size_t)L.inner * L.dtp));
      TRY(W(&L.w_uv, (size_t)L.n_x * L.inner));
      TRY(W(&L.w_o, D * L.inner));
      TRY(F(&L.f_a, (size_t)L.inner * L.nstate));
      TRY(F(&L.f_b, L.inner));
      TRY(F(&L.f_c, L.inner));
      TRY(F(&L.conv, (size_t)L.inner * L.taps));
      TRY(F(&L.conv_b, L.inner));
      need({"mix.in", "mix.conv", "mix.conv.b", "mix.x", "mix.dt", "mix.dt.b", "mix.A_log", "mix.D"});
    } else {
      TRY(W(&L.w_uk, (size_t)L.H * L.d * L.rap));
      TRY(W(&L.w_uv, (size_t)L.H * L.vd * L.rgp));
      TRY(W(&L.w_o, D * L.H * L.vd));
      TRY(F(&L.f_a, L.vd));
      TRY(F(&L.f_b, L.H));
      TRY(F(&L.f_c, (size_t)L.H * L.d));
      TRY(F(&L.conv, (size_t)L.conv_ch() * L.taps));
      need({"mix.q", "mix.q.conv", "mix.k", "mix.k.conv", "mix.v", "mix.v.conv", "mix.b", "mix.A_log", "mix.norm", "mix.a1",
            "mix.a2", "mix.dt_bias", "mix.g1", "mix.g2"});
    }
    if (L.ff) {
      const bool stacked = L.ff_plain && hm.res_gate;          // up | gate of the result: both read the same rows
      const size_t n = std::max(1, L.n_mats());
      TRY(F(&L.norm2, D));
      TRY(W(&L.w_gu, n * (L.single_up() ? L.ffp + (stacked ? D : 0) : 2 * L.ffp) * D));
      TRY(W(&L.w_down, n * D * L.ffp));
      need({"norm2"});
      if (L.n_exp) {
        TRY(W(&L.w_router, (size_t)L.n_router() * D));
        need({"mlp.router"});
        if (L.sff) {
          if (L.joined()) {
            L.w_sgu = (char*)L.w_gu + (size_t)L.n_exp * 2 * L.ffp * D * e;
            L.w_sdown = (char*)L.w_down + (size_t)L.n_exp * D * L.ffp * e;
          } else {
            TRY(W(&L.w_sgu, (size_t)2 * L.sffp * D));
            TRY(W(&L.w_sdown, D * L.sffp));
          }
          need({"mlp.shared.gate", "mlp.shared.up", "mlp.shared.down", "mlp.shared.sg"});
        }
        if (L.corrected) { TRY(F(&L.correction, L.n_out())); need({"mlp.correction"}); }
        for (int x = 0; x < L.n_exp; ++x)
          for (const char* part : {".gate", ".up", ".down"}) hm.want.insert(p + "mlp.e" + std::to_string(x) + part);
      } else {
        need({"mlp.up", "mlp.down"});
        if (!L.single_up()) need({"mlp.gate"});
        if (L.poly) { TRY(F(&L.coef, 4)); need({"mlp.act"}); }
      }
      if (stacked) L.w_rg[1] = (char*)L.w_gu + (size_t)L.ffp * D * e;
    }
    if (hm.side) {
      TRY(W(&L.w_sgate, (size_t)up4(hm.side) * D));
      TRY(W(&L.w_sproj, D * hm.sidep));
      TRY(F(&L.s_norm, D));
      need({"side.gate", "side.proj", "side.norm"});
    }
    for (int q = 0; q < (L.ff ? 2 : 1); ++q) {
      const std::string k = std::to_string(q + 1);
      if (hm.post_norm) {
        TRY(F(&L.post[q], D));
        hm.want.insert(p + "norm" + k + "b");
      }
      if (hm.streams) {
        TRY(F(&L.hc_in[q], hm.streams));
        TRY(F(&L.hc_out[q], hm.streams));
        TRY(F(&L.hc_mix[q], hm.streams * hm.streams));
        for (const char* part : {".in", ".out", ".mix"}) hm.want.insert(p + "hc" + k + part);
      }
      if (hm.res_gate) {
        if (!L.w_rg[q]) TRY(W(&L.w_rg[q], D * D));
        TRY(F(&L.rg_b[q], D));
        hm.want.insert(p + "rg" + k);
        hm.want.insert(p + "rg" + k + ".b");
      }
    }
    if (hm.in_taps) {
      TRY(F(&L.in_conv, D * hm.in_taps));
      need({"canon1"});
    }
  }
  return VN_OK;
}

void destroy(vn_model* m) {
  if (!m->hyb) return;
  auto F = [](void* p) { if (p) cudaFree(p); };
  Model& hm = *m->hyb;
  for (auto& L : hm.layers) {
    F(L.norm1); F(L.norm2); F(L.w_in); F(L.w_o); F(L.w_uk); F(L.w_uv); F(L.f_a); F(L.f_b); F(L.f_c); F(L.conv); F(L.conv_b);
    if (!(L.ff_plain && hm.res_gate)) F(L.w_rg[1]);            // else part of w_gu
    F(L.w_gu); F(L.w_down); F(L.w_rg[0]); F(L.in_conv);
    F(L.f_d); F(L.o_b); F(L.w_router); F(L.correction); F(L.w_sgate); F(L.w_sproj); F(L.s_norm);
    F(L.temp); F(L.coef);
    if (!L.joined()) { F(L.w_sgu); F(L.w_sdown); }             // else part of w_gu, w_down
    for (int q = 0; q < 2; ++q) { F(L.post[q]); F(L.hc_in[q]); F(L.hc_out[q]); F(L.hc_mix[q]); F(L.rg_b[q]); }
  }
  for (Rope& r : hm.ropes) F(r.table);
  for (void* t : hm.retired) F(t);
  F(hm.w_loop); F(hm.loop_step); F(hm.freq); F(hm.x0); F(hm.cat); F(hm.ws); F(hm.meta);
  F(hm.hc); F(hm.gate); F(hm.y); F(hm.gate_ws); F(hm.seg);
  F(hm.side_embed); F(hm.exp_count); F(hm.exp_cur); F(hm.exp_off);
  delete m->hyb;
  m->hyb = nullptr;
}

// ---- weights: checkpoint names to their places in the stacked, padded matrices -----------------------------------
int32_t load(vn_model* m, const std::string& n, const float* data, long long r, long long cl) {
  vn_ctx* ctx = m->ctx;
  Model& hm = *m->hyb;
  const long long D = hm.D;
  int32_t st = VN_OK;
  // expected shape; a vector is (n, 1)
  auto shape = [&](long long er, long long ec) -> bool {
    if (r == er && cl == ec) return true;
    st = vn_fail(ctx, VN_ERR_INVALID, "%s: shape (%lld, %lld) expected (%lld, %lld)", n.c_str(), r, cl, er, ec);
    return false;
  };
  auto rows = [&](void* dst, long long ld, long long row_off = 0, long long row_mul = 1) {
    return upload(m, data, dst, r, cl, ld, row_mul, row_off);
  };
  auto f32 = [&](const float* src, float* dst, long long count) { return upload(m, src, dst, 1, count, count, 1, 0, true); };
  std::vector<float> tmp;
  auto mapped = [&](float* dst, long long count, float (*fn)(float)) {
    tmp.resize(count);
    for (long long i = 0; i < count; ++i) tmp[i] = fn(data[i]);
    return f32(tmp.data(), dst, count);
  };
  auto one_plus = [](float w) { return 1.0f + w; };
  auto rate = [](float a) { return expf(a); };
  auto neg_rate = [](float a) { return -expf(a); };
  if (!hm.want.count(n)) {
    // a layer without a feed-forward has no use for its second sublayer's tensors
    const size_t at = n.find('.');
    const int i = n[0] == 'l' && at != std::string::npos ? atoi(n.substr(1, at - 1).c_str()) : -1;
    const std::string part = at != std::string::npos ? n.substr(at + 1) : "";
    if (i >= 0 && i < (int)hm.layers.size() && !hm.layers[i].ff && n.substr(0, at) == "l" + std::to_string(i) &&
        (part == "norm2" || part == "norm2b" || part.compare(0, 4, "hc2.") == 0 || part == "rg2" || part == "rg2.b"))
      return VN_OK;
    return vn_fail(ctx, VN_ERR_INVALID, "unexpected tensor %s", n.c_str());
  }
  auto weight = [&](float* dst, long long count) {        // a norm's: around zero or plain
    return hm.plain_norm ? f32(data, dst, count) : mapped(dst, count, one_plus);
  };
#define PUT(er, ec, expr) do { if (!shape((er), (ec))) return st; TRY(expr); return VN_OK; } while (0)
  if (n == "embed") PUT(hm.vocab, D, rows(m->emb, D));
  if (n == "head") PUT(hm.vocab, D, rows(m->head, D));
  if (n == "final.norm") PUT(D, 1, weight(m->norm_f, D));
  if (n == "side.embed") PUT(hm.vocab, (long long)hm.layers.size() * hm.side, rows(hm.side_embed, cl));
  if (n == "loop.in") PUT(D, 2 * D, rows(hm.w_loop, 2 * D));
  if (n == "loop.step") PUT(hm.loop_times, D, f32(data, hm.loop_step, r * cl));
  const size_t dot = n.find('.');
  HLayer& L = hm.layers[atoi(n.substr(1, dot - 1).c_str())];      // the name is in `want`: the layer exists
  const std::string s = n.substr(dot + 1);
  if (s == "norm1") PUT(D, 1, weight(L.norm1, D));
  if (s == "norm2") PUT(D, 1, weight(L.norm2, D));
  if (s == "norm1b") PUT(D, 1, weight(L.post[0], D));
  if (s == "norm2b") PUT(D, 1, weight(L.post[1], D));
  if (s == "mlp.act") PUT(4, 1, f32(data, L.coef, 4));
  if (s == "mlp.gate") PUT(L.ff, D, rows(L.w_gu, D, 0, 2));
  if (s == "mlp.up" && L.single_up()) PUT(L.ff, D, rows(L.w_gu, D));
  if (s == "mlp.up") PUT(L.ff, D, rows(L.w_gu, D, 1, 2));
  if (s == "mlp.down") PUT(D, L.ff, rows(L.w_down, L.ffp));
  if (s == "mlp.router") PUT(L.n_out(), D, rows(L.w_router, D));
  if (s == "mlp.shared.sg") PUT(1, D, rows(L.w_router, D, L.n_out()));
  if (s == "mlp.shared.gate") PUT(L.sff, D, rows(L.w_sgu, D, 0, 2));
  if (s == "mlp.shared.up") PUT(L.sff, D, rows(L.w_sgu, D, 1, 2));
  if (s == "mlp.shared.down") PUT(D, L.sff, rows(L.w_sdown, L.sffp));
  if (s == "mlp.correction") PUT(L.n_out(), 1, f32(data, L.correction, r));
  if (s.compare(0, 5, "mlp.e") == 0) {
    const size_t end = s.find('.', 4);
    const long long x = atoll(s.substr(5, end - 5).c_str());
    const std::string part = s.substr(end + 1);
    void* gu = (char*)L.w_gu + x * 2 * L.ffp * D * m->esz;
    if (part == "gate") PUT(L.ff, D, rows(gu, D, 0, 2));
    if (part == "up") PUT(L.ff, D, rows(gu, D, 1, 2));
    PUT(D, L.ff, rows((char*)L.w_down + x * D * L.ffp * m->esz, L.ffp));
  }
  if (s == "side.gate") PUT(hm.side, D, rows(L.w_sgate, D));
  if (s == "side.proj") PUT(D, hm.side, rows(L.w_sproj, hm.sidep));
  if (s == "side.norm") PUT(D, 1, f32(data, L.s_norm, r));
  if (s == "canon1") PUT(D, hm.in_taps, f32(data, L.in_conv, r * cl));
  for (int q = 0; q < 2; ++q) {
    const std::string k = std::to_string(q + 1);
    if (s == "hc" + k + ".in") PUT(hm.streams, 1, f32(data, L.hc_in[q], r));
    if (s == "hc" + k + ".out") PUT(hm.streams, 1, f32(data, L.hc_out[q], r));
    if (s == "hc" + k + ".mix") PUT(hm.streams, hm.streams, f32(data, L.hc_mix[q], r * cl));
    if (s == "rg" + k) PUT(D, D, rows(L.w_rg[q], D));
    if (s == "rg" + k + ".b") PUT(D, 1, f32(data, L.rg_b[q], D));
  }
  if (L.kind == ATTENTION) {
    const long long qd = (long long)L.H * L.d, kd = (long long)L.KH * L.d, vd = (long long)L.KH * L.vd, hv = (long long)L.H * L.vd;
    if (s == "mix.q") PUT(qd, D, rows(L.w_in, D));
    if (s == "mix.k") PUT(kd, D, rows(L.w_in, D, qd));
    if (s == "mix.v") PUT(vd, D, rows(L.w_in, D, qd + kd));
    if (s == "mix.g") PUT(L.attn_gates(), D, rows(L.w_in, D, L.conv_ch()));
    if (s == "mix.temp") PUT(L.H, 1, f32(data, L.temp, r));
    if (s == "mix.q.norm") PUT(L.d, 1, f32(data, L.f_a, r));
    if (s == "mix.k.norm") PUT(L.d, 1, f32(data, L.f_b, r));
    if (s == "mix.q.b") PUT(qd, 1, f32(data, L.f_c, r));
    if (s == "mix.k.b") PUT(kd, 1, f32(data, L.f_c + qd, r));
    if (s == "mix.v.b") PUT(vd, 1, f32(data, L.f_c + qd + kd, r));
    if (s == "mix.o.b") PUT(D, 1, f32(data, L.o_b, r));
    if (s == "mix.q.conv") PUT(qd, L.taps, f32(data, L.conv, r * cl));
    if (s == "mix.k.conv") PUT(kd, L.taps, f32(data, L.conv + qd * L.taps, r * cl));
    if (s == "mix.v.conv") PUT(vd, L.taps, f32(data, L.conv + (qd + kd) * L.taps, r * cl));
    if (s == "mix.o") PUT(D, hv, rows(L.w_o, hv));
  } else if (L.kind == LIGHTNING) {
    const long long qd = (long long)L.H * L.d, hv = (long long)L.H * L.vd;
    if (s == "mix.q") PUT(qd, D, rows(L.w_in, D));
    if (s == "mix.k") PUT(qd, D, rows(L.w_in, D, qd));
    if (s == "mix.v") PUT(hv, D, rows(L.w_in, D, 2 * qd));
    if (s == "mix.g") PUT(hv, D, rows(L.w_in, D, 2 * qd + hv));
    if (s == "mix.norm") PUT(hv, 1, f32(data, L.f_a, r));
    if (s == "mix.o") PUT(D, hv, rows(L.w_o, hv));
  } else if (L.kind == LATENT) {
    const long long hd = (long long)L.H * L.d, hv = (long long)L.H * L.vd, hq = hd + (long long)L.H * L.rr;
    if (s == "mix.q") PUT(hq, D, rows(L.w_in, D));
    if (s == "mix.dkv") PUT(L.R + L.rr, D, rows(L.w_in, D, hq));
    if (s == "mix.g") PUT(L.n_gate(), D, rows(L.w_in, D, hq + L.R + L.rr));
    if (s == "mix.dkv.norm") PUT(L.R, 1, f32(data, L.f_a, L.R));
    if (s == "mix.sink") PUT(L.H, 1, f32(data, L.f_b, L.H));
    if (s == "mix.uv") PUT(hv, L.R, rows(L.w_uv, L.Rp));
    if (s == "mix.o") PUT(D, hv, rows(L.w_o, hv));
    if (s == "mix.uk") {          // stored per head as [d, R], used as its transpose
      if (!shape(hd, L.R)) return st;
      tmp.assign((size_t)L.H * L.Rp * L.dp, 0.f);
      for (long long h = 0; h < L.H; ++h)
        for (long long i = 0; i < L.d; ++i)
          for (long long c = 0; c < L.R; ++c) tmp[(h * L.Rp + c) * L.dp + i] = data[(h * L.d + i) * L.R + c];
      return upload(m, tmp.data(), L.w_uk, (long long)L.H * L.Rp, L.dp, L.dp);
    }
  } else if (L.kind == MAMBA2) {
    const long long C = L.conv_ch();
    if (s == "mix.in") PUT(L.inner + C + L.H, D, rows(L.w_in, D));
    if (s == "mix.conv") PUT(C, L.taps, f32(data, L.conv, r * cl));
    if (s == "mix.conv.b") PUT(C, 1, f32(data, L.conv_b, r));
    if (s == "mix.dt_bias") PUT(L.H, 1, f32(data, L.f_c, r));
    if (s == "mix.A_log") PUT(L.H, 1, mapped(L.f_d, r, neg_rate));
    if (s == "mix.D") PUT(L.H, 1, f32(data, L.f_b, r));
    if (s == "mix.norm") PUT(L.inner, 1, f32(data, L.f_a, r));
    if (s == "mix.o") PUT(D, L.inner, rows(L.w_o, L.inner));
  } else if (L.kind == MAMBA1) {
    if (s == "mix.in") PUT(2ll * L.inner, D, rows(L.w_in, D));
    if (s == "mix.conv") PUT(L.inner, L.taps, f32(data, L.conv, r * cl));
    if (s == "mix.conv.b") PUT(L.inner, 1, f32(data, L.conv_b, r));
    if (s == "mix.x") {           // dt rows first, B and C behind the padded dt block
      if (!shape(L.dt_rank + 2ll * L.nstate, L.inner)) return st;
      TRY(upload(m, data, L.w_uv, L.dt_rank, L.inner, L.inner));
      return upload(m, data + (long long)L.dt_rank * L.inner, L.w_uv, 2ll * L.nstate, L.inner, L.inner, 1, L.dtp);
    }
    if (s == "mix.dt") PUT(L.inner, L.dt_rank, rows(L.w_uk, L.dtp));
    if (s == "mix.dt.b") PUT(L.inner, 1, f32(data, L.f_c, r));
    if (s == "mix.A_log") PUT(L.inner, L.nstate, mapped(L.f_a, r * cl, neg_rate));
    if (s == "mix.D") PUT(L.inner, 1, f32(data, L.f_b, r));
    if (s == "mix.o") PUT(D, L.inner, rows(L.w_o, L.inner));
  } else {
    const long long kd = (long long)L.KH * L.d, hv = (long long)L.H * L.vd, b0 = 2 * kd + hv;
    if (s == "mix.q") PUT(kd, D, rows(L.w_in, D));
    if (s == "mix.k") PUT(kd, D, rows(L.w_in, D, kd));
    if (s == "mix.v") PUT(hv, D, rows(L.w_in, D, 2 * kd));
    if (s == "mix.b") PUT(L.H, D, rows(L.w_in, D, b0));
    if (s == "mix.a1") PUT(L.ra, D, rows(L.w_in, D, b0 + L.H));
    if (s == "mix.g1") PUT(L.rg, D, rows(L.w_in, D, b0 + L.H + L.ra));
    if (s == "mix.q.conv") PUT(kd, L.taps, f32(data, L.conv, r * cl));
    if (s == "mix.k.conv") PUT(kd, L.taps, f32(data, L.conv + kd * L.taps, r * cl));
    if (s == "mix.v.conv") PUT(hv, L.taps, f32(data, L.conv + 2 * kd * L.taps, r * cl));
    if (s == "mix.a2") PUT((long long)L.H * L.d, L.ra, rows(L.w_uk, L.rap));
    if (s == "mix.g2") PUT(hv, L.rg, rows(L.w_uv, L.rgp));
    if (s == "mix.A_log") PUT(L.H, 1, mapped(L.f_b, r, rate));
    if (s == "mix.dt_bias") PUT((long long)L.H * L.d, 1, f32(data, L.f_c, r));
    if (s == "mix.norm") PUT(L.vd, 1, f32(data, L.f_a, r));
    if (s == "mix.o") PUT(D, hv, rows(L.w_o, hv));
  }
#undef PUT
  return vn_fail(ctx, VN_ERR_INVALID, "unexpected tensor %s", n.c_str());
}

int32_t finalize(vn_model* m) {
  for (auto& w : m->hyb->want)
    if (!m->loaded.count(w)) return vn_fail(m->ctx, VN_ERR_INVALID, "missing tensor %s", w.c_str());
  m->finalized = true;
  return VN_OK;
}

// ---- activations ---------------------------------------------------------------------------------------------------
int32_t ensure(vn_model* m, int M) {
  if (M <= m->cap_rows) return VN_OK;
  vn_ctx* ctx = m->ctx;
  Model& hm = *m->hyb;
  VN_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
  m->cap_rows = 0;
  void** bufs[] = {(void**)&m->x, &m->h, (void**)&hm.x0, &hm.cat, (void**)&hm.ws, &hm.hc, (void**)&hm.gate, (void**)&hm.y};
  for (void** b : bufs) { if (*b) cudaFree(*b); *b = nullptr; }
  const size_t R = (size_t)M + (M >> 2) + 32, D = hm.D, e = m->esz;
  TRY(dev_alloc(ctx, (void**)&m->x, R * D * 4 * std::max(1, hm.streams)));
  TRY(dev_alloc(ctx, &m->h, R * D * e));
  if (hm.arranged || hm.loop_times) TRY(dev_alloc(ctx, (void**)&hm.x0, R * D * 4));
  if (hm.arranged) {
    TRY(dev_alloc(ctx, &hm.hc, R * D * e));
    TRY(dev_alloc(ctx, (void**)&hm.gate, R * D * 4));
    TRY(dev_alloc(ctx, (void**)&hm.y, R * D * 4));
  }
  if (hm.loop_times && !hm.loop_add) TRY(dev_alloc(ctx, &hm.cat, R * 2 * D * e));
  size_t need = 0;
  for (auto& L : hm.layers)
    for (size_t rows : {R, std::min(R, (size_t)SPLIT_ROWS)}) {
      Arena A;
      Buffers b;
      layout(hm, L, rows, e, A, b);
      need = std::max(need, A.off);
    }
  TRY(dev_alloc(ctx, (void**)&hm.ws, need));
  hm.ws_bytes = need;
  m->cap_rows = (int)R;
  return VN_OK;
}

// ---- projections -----------------------------------------------------------------------------------------------------
bool tc_rows(const vn_model* m, const GemmArgs& g) {
  return m->cfg.bf16 && m->use_tc && g.M <= 256 && g.N % 4 == 0 && gemm_tc_supported(g);
}
GemmArgs gemm_args(const void* A, int lda, const void* W, int N, int K, int M, const char* tag) {
  GemmArgs g;
  g.A = A; g.lda = lda; g.W = W; g.ldw = K; g.M = M; g.N = N; g.K = K; g.tag = tag;
  return g;
}
// out = A W^T in fp32: split-K slices in the workspace, or the matrix `direct`
int32_t project(vn_model* m, GemmArgs g, float* direct, Src* out, bool gate = false) {
  *out = Src();
  out->ld = g.N;
  if (tc_rows(m, g)) {
    int sp = 1;
    // a gate's slices outlive the projections that follow it: they have a workspace of their own
    auto other = [&] { if (gate) { std::swap(m->partial, m->hyb->gate_ws); std::swap(m->partial_bytes, m->hyb->gate_ws_bytes); } };
    other();
    const int32_t st = tc_partial(m, g, g.M, g.M, &sp);
    out->p = m->partial; out->splits = sp; out->pstride = (long long)g.M * g.N;
    other();
    return st;
  }
  g.C = direct; g.ldc = g.N;
  out->p = direct;
  return linear(m, g);
}
// the same in 16 bits (many rows), with the GEMM's own function on some columns
int32_t project(vn_model* m, GemmArgs g, float* direct, Mat<__nv_bfloat16>* out, bool = false) {
  g.C = direct; g.ldc = g.N; g.c_bf16 = 1;
  out->p = (const __nv_bfloat16*)direct; out->ld = g.N;
  return linear(m, g);
}
// what follows a sublayer: the entry of a looped block's pass, and in m->h RMSNorm(x) * norm_w, x itself, or nothing
struct Next { const float* norm_w = nullptr; bool cast = false; PassEntry pass; };

// x += y (or y over its root mean square times own_norm), and what the next product reads, in one pass over the rows
template <typename T, typename Y>
int32_t close_rows(vn_model* m, const Y& y, int M, const float* own_norm, const Next& next) {
  vn_ctx* ctx = m->ctx;
  const int D = m->hyb->D;
  const float eps = m->hyb->eps;
#define RESIDUAL(NV) VN_LAUNCH_PDL_LEVEL(ctx, 1, "residual_kernel", (residual_kernel<T, Y, NV>), M, 256, 0, y, m->x, own_norm, next.pass, next.norm_w, (int)next.cast, (T*)m->h, D, eps)
  if (D % 4 || D > 8192) RESIDUAL(0); else if (D <= 1024) RESIDUAL(1); else if (D <= 2048) RESIDUAL(2); else if (D <= 4096) RESIDUAL(4); else RESIDUAL(8);
#undef RESIDUAL
  return VN_OK;
}

// x += A W^T over its root mean square times own_norm; then as `next` says.  direct: [M, D] fp32 scratch
template <typename T>
int32_t close_normed(vn_model* m, const GemmArgs& g, const float* bias, float* direct, const float* own_norm, const Next& next) {
  if constexpr (std::is_same<T, __nv_bfloat16>::value)
    if (g.M > 256) {
      AddRows<Mat<T>> y;
      y.bias = bias;
      TRY(project(m, g, direct, &y.y));
      return close_rows<T>(m, y, g.M, own_norm, next);
    }
  AddRows<Src> y;
  y.bias = bias;
  TRY(project(m, g, direct, &y.y));
  return close_rows<T>(m, y, g.M, own_norm, next);
}

// x += A W^T (+ bias); then as `next` says
template <typename T>
int32_t close_block(vn_model* m, GemmArgs g, const float* bias, const Next& next) {
  vn_ctx* ctx = m->ctx;
  const Model& hm = *m->hyb;
  const int D = hm.D, M = g.M;
  const float* next_norm = next.norm_w;
  if (tc_rows(m, g)) {
    int sp = 1;
    TRY(tc_partial(m, g, M, M, &sp));
    if (bias || next.cast || next.pass.step) {
      AddRows<Src> y;
      y.y.p = m->partial; y.y.splits = sp; y.y.pstride = (long long)M * D; y.y.ld = D; y.bias = bias;
      return close_rows<T>(m, y, M, nullptr, next);
    }
    if (D % 4 == 0 && D <= 2048) {
      VN_LAUNCH_PDL_BIT(ctx, 4, splitk_add_norm_kernel<T>, M, 256, 0, m->partial, sp, (long long)M * D, m->x, next_norm,
                        (T*)m->h, (float*)nullptr, D, hm.eps);
    } else {
      Src s;
      s.p = m->partial; s.splits = sp; s.pstride = (long long)M * D; s.ld = D;
      VN_LAUNCH(ctx, rowsum_norm_kernel<T>, M, 256, 0, s, (const float*)nullptr, 1, m->x, next_norm, (T*)m->h, D, hm.eps);
    }
    return VN_OK;
  }
  g.C = m->x; g.ldc = D; g.epi = EPI_ADD; g.bias = bias;
  TRY(linear(m, g));
  if (next.cast) {
    const long long n = (long long)M * D;
    VN_LAUNCH(ctx, cast_rows_kernel<T>, (unsigned)ceil_div(n, 1024ll), 256, 0, m->x, (T*)m->h, n);
  }
  if (next.pass.step)
    VN_LAUNCH(ctx, enter_pass_kernel<T>, M, 256, 0, next.pass, m->x, next_norm, (T*)m->h, D, hm.eps);
  else if (next_norm)
    VN_LAUNCH(ctx, rmsnorm_kernel<T>, M, 256, 0, m->x, next_norm, (T*)m->h, (float*)nullptr, 1, 0, D, hm.eps);
  return VN_OK;
}
// nseg products of equal shape, one per head
int32_t batched(vn_model* m, const GemmArgs& g) {
  if (m->cfg.bf16 && gemm_mma_supported(g)) return launch_gemm_mma(m->ctx, g);
  if (m->cfg.bf16) return launch_gemm_simt<__nv_bfloat16, __nv_bfloat16>(m->ctx, g);
  return launch_gemm_simt<float, float>(m->ctx, g);
}

// ---- mixers: normalised rows -> the input of the output projection -----------------------------------------------------------
// S: Src, or the 16-bit matrix of a forward of many rows
template <typename T, typename S>
int32_t latent_attention(vn_model* m, const void* in_rows, vn_kv* kv, Cache& hc, const HLayer& L, int run, const Rows& rows, const Buffers& b) {
  vn_ctx* ctx = m->ctx;
  const int M = rows.M, D = m->hyb->D, H = L.H;
  S s;
  TRY(project(m, gemm_args(in_rows, D, L.w_in, L.n_in, D, M, "gemm_latent_in"), b.proj, &s));
  LatentIn in;
  in.H = H; in.d = L.d; in.dp = L.dp; in.rr = L.rr; in.R = L.R; in.Rp = L.Rp; in.rope = L.rope >= 0 ? m->hyb->ropes[L.rope].table : nullptr;
  in.norm_w = L.f_a; in.eps = m->hyb->eps; in.n_gate = L.n_gate(); in.gate = b.gate; in.gate_t = b.gate_t;
  in.q = b.q; in.qc = b.qc; in.plane = kv->k[run]; in.table = hc.table_dev; in.max_pages = hc.max_pages;
  const int parts = M > 256 ? 1 : std::min(16, ceil_div(L.n_in, 512));
  VN_LAUNCH_NAMED(ctx, "latent_append_kernel", (latent_append_kernel<T, S>), dim3(M, parts), 256, (size_t)L.R * 4, s, in, rows);
  GemmArgs g = gemm_args(b.q, H * L.dp, L.w_uk, L.rr ? L.R : L.Rp, L.dp, M, "gemm_latent_uk");
  g.C = b.qc; g.ldc = (long long)H * L.Rp; g.c_bf16 = m->cfg.bf16;
  g.nseg = H; g.a_stride = L.dp; g.w_stride = (long long)L.Rp * L.dp; g.c_stride = L.Rp;
  TRY(batched(m, g));
  LatentArgs a;
  a.qc = b.qc; a.plane = kv->k[run]; a.table = hc.table_dev; a.max_pages = hc.max_pages; a.Rp = L.Rp; a.H = H;
  a.window = L.window; a.scale = L.scale; a.sink = L.sinks ? L.f_b : nullptr; a.gate = b.gate; a.out = b.oc; a.rows = rows;
  const bool mma = m->cfg.bf16 && L.Rp <= 576 && !m->force_simt_attn;
  if (mma && M <= SPLIT_ROWS) {       // few rows: several CTAs share a tile's key pages
    const int tile = latent_tile_rows(L.Rp, rows.max_n * H), tiles = rows.n_ent * ceil_div(rows.max_n * H, tile);
    const int pages = L.window > 0 ? std::min(hc.max_pages, (L.window + rows.max_n) / KV_PAGE + 2) : hc.max_pages;
    a.splits = std::max(1, std::min(std::min(MAX_SPLITS, pages / 2), 2 * ctx->sm_count / std::max(1, tiles)));
    a.part_o = b.part_o; a.part_ml = b.part_ml;
  }
  TRY(vn_latent_attention(ctx, a, m->cfg.bf16 != 0, mma));
  g = gemm_args(b.oc, H * L.Rp, L.w_uv, L.vd, L.Rp, M, "gemm_latent_uv");
  g.C = b.mix; g.ldc = (long long)H * L.vd; g.c_bf16 = m->cfg.bf16;
  g.nseg = H; g.a_stride = L.Rp; g.w_stride = (long long)L.vd * L.Rp; g.c_stride = L.vd; g.mul = b.gate_t;
  return batched(m, g);
}

template <typename T>
ConvIn<T> conv_in(const HLayer& L, const Cache& hc, const Src& s, void* ring) {
  ConvIn<T> c;
  c.src = s; c.ring = (T*)ring; c.RC = L.taps - 1 + hc.pending; c.C = L.conv_ch(); c.taps = L.taps; c.w = L.conv; c.bias = L.conv_b;
  return c;
}

int32_t ensure_segments(vn_model* m, size_t bytes) {
  Model& hm = *m->hyb;
  if (bytes <= hm.seg_bytes) return VN_OK;
  VN_CUDA(m->ctx, cudaStreamSynchronize(m->ctx->stream));
  if (hm.seg) cudaFree(hm.seg);
  hm.seg = nullptr; hm.seg_bytes = 0;
  TRY(dev_alloc(m->ctx, (void**)&hm.seg, bytes));
  hm.seg_bytes = bytes;
  return VN_OK;
}

template <typename T>
int32_t mamba1(vn_model* m, const void* in_rows, vn_kv* kv, Cache& hc, const HLayer& L, int run, const Rows& rows, const Buffers& b) {
  vn_ctx* ctx = m->ctx;
  const int M = rows.M, D = m->hyb->D, n = L.inner;
  Src s;
  TRY(project(m, gemm_args(in_rows, D, L.w_in, L.n_in, D, M, "gemm_mamba_in"), b.proj, &s));
  const ConvIn<T> cv = conv_in<T>(L, hc, s, kv->k[run]);
  if (rows.max_n == 1)
    VN_LAUNCH(ctx, (mamba_conv_kernel<T, 1>), dim3(ceil_div(n, 32), ceil_div(M, 8)), dim3(32, 8), 0, cv, rows, (T*)b.xc, (T*)b.z, hc.pending);
  else
    VN_LAUNCH(ctx, (mamba_conv_kernel<T, 8>), dim3(ceil_div(n, 32), ceil_div(M, 64)), dim3(32, 8), 0, cv, rows, (T*)b.xc, (T*)b.z, hc.pending);
  if (rows.max_n > hc.pending)
    VN_LAUNCH(ctx, (conv_tail_kernel<T, Src, true>), dim3(ceil_div(n, 256), rows.n_ent), 256, 0, cv, rows, hc.pending);
  MambaArgs a;
  TRY(project(m, gemm_args(b.xc, n, L.w_uv, L.n_x, n, M, "gemm_mamba_x"), b.p, &a.p));
  a.xc = b.xc; a.z = b.z; a.dt_cols = L.dtp; a.dt_rank = L.dt_rank; a.w_dt = L.w_uk; a.dt_bias = L.f_c; a.A = L.f_a; a.D = L.f_b;
  a.state = (float*)kv->v[run]; a.R = hc.ring_len; a.inner = n; a.nstate = L.nstate; a.out = b.mix; a.rows = rows;
  if (rows.max_n == 1) {
    if (M >= 16 && a.p.splits > 1) {     // many rows: the slices are summed once, not by every CTA of a row
      VN_LAUNCH(ctx, splitk_store_kernel, (unsigned)ceil_div((long long)M * L.n_x, 256ll), 256, 0, a.p.p, a.p.splits, a.p.pstride,
                b.p, (long long)L.n_x, L.n_x, (long long)M * L.n_x);
      a.p = Src();
      a.p.p = b.p; a.p.ld = L.n_x;
    }
    TRY(vn_mamba_step(ctx, a, m->cfg.bf16 != 0));
    return VN_OK;
  }
  VN_LAUNCH(ctx, cast_cols_kernel<T>, M, 64, 0, a.p, 0, L.dt_rank, (T*)b.dtb, L.dtp);
  GemmArgs g = gemm_args(b.dtb, L.dtp, L.w_uk, n, L.dtp, M, "gemm_mamba_dt");
  g.C = b.dt; g.ldc = n;
  TRY(linear(m, g));
  a.dt = b.dt;
  return vn_mamba_scan(ctx, a, m->cfg.bf16 != 0);
}

// S: Src, or the 16-bit matrix of a forward of many rows
template <typename T, typename S>
int32_t mamba2(vn_model* m, const void* in_rows, vn_kv* kv, Cache& hc, const HLayer& L, int run, const Rows& rows, const Buffers& b) {
  vn_ctx* ctx = m->ctx;
  Model& hm = *m->hyb;
  const int M = rows.M, D = hm.D;
  ConvIn<T, S> cv;
  TRY(project(m, gemm_args(in_rows, D, L.w_in, L.n_in, D, M, "gemm_ssd_in"), b.proj, &cv.src));
  cv.col0 = L.inner; cv.ring = (T*)kv->k[run]; cv.RC = L.taps - 1 + hc.pending; cv.C = L.conv_ch(); cv.taps = L.taps; cv.w = L.conv; cv.bias = L.conv_b;
  SsdArgs a;
  a.H = L.H; a.P = L.vd; a.N = L.nstate; a.G = L.groups; a.xbc = b.xbc; a.ld = up8(L.conv_ch()); a.dt = b.dt; a.dt_bias = L.f_c; a.A = L.f_d; a.D = L.f_b;
  a.state = (float*)kv->v[run]; a.R = hc.ring_len; a.pending = hc.pending; a.u = b.u; a.rows = rows;
  bool step = false;
  if constexpr (std::is_same<S, Src>::value) {
    step = rows.max_n == 1 && M < SSD_STEP_ROWS;      // few rows: one kernel; many: each row's inputs are convolved only once
    if (step) TRY(vn_ssd_step<T>(ctx, cv, a));
    else if (rows.max_n == 1) a.z = b.z;
  }
  if (!step) {
    TRY((vn_ssd_inputs<T, S>(ctx, cv, a)));
    if (rows.max_n > hc.pending && L.taps > 1)
      VN_LAUNCH(ctx, (conv_tail_kernel<T, S, true>), dim3(ceil_div(cv.C, 256), rows.n_ent), 256, 0, cv, rows, hc.pending);
    const SsdPlan plan = vn_ssd_plan(ctx, m->cfg.bf16 != 0, L.H, L.nstate, L.vd, rows, hc.pending);
    if (plan.chunked) {
      if constexpr (std::is_same<T, __nv_bfloat16>::value) {
        TRY(ensure_segments(m, plan.seg_bytes));
        a.segments = plan.segments; a.seg_len = plan.seg_len; a.seg_state = hm.seg;
        a.seg_decay = hm.seg + (long long)rows.n_ent * plan.segments * L.H * L.nstate * L.vd;
        TRY(vn_ssd_chunks(ctx, cv.src, a));
      }
    } else {
      TRY((vn_ssd_scan<T, S>(ctx, cv.src, a)));
    }
  }
  return vn_ssd_norm<T>(ctx, (const T*)b.u, L.f_a, (T*)b.mix, M, L.inner, L.norm_groups, hm.eps);
}

template <typename T>
int32_t channel_delta(vn_model* m, const void* in_rows, vn_kv* kv, Cache& hc, const HLayer& L, int run, const Rows& rows, const Buffers& b) {
  vn_ctx* ctx = m->ctx;
  const int M = rows.M, D = m->hyb->D, H = L.H, KH = L.KH, d = L.d, vd = L.vd;
  Src s;
  TRY(project(m, gemm_args(in_rows, D, L.w_in, L.n_in, D, M, "gemm_delta_in"), b.proj, &s));
  const ConvIn<T> cv = conv_in<T>(L, hc, s, kv->k[run]);
  DeltaIn in;
  in.src = s; in.H = H; in.KH = KH; in.d = d; in.vd = vd; in.ra = L.ra; in.rg = L.rg; in.ra_ld = L.rap; in.rg_ld = L.rgp;
  in.col_b = 2 * KH * d + H * vd; in.col_a = in.col_b + H; in.col_g = in.col_a + L.ra;
  in.q = b.dq; in.k = b.dk; in.v = b.dv; in.beta = b.beta; in.low_a = b.low_a; in.low_g = b.low_g;
  in.rows = rows; in.pending = hc.pending;
  if (rows.max_n == 1) {
    DeltaStepArgs<T> a;
    a.conv = cv; a.in = in; a.w_a = (const T*)L.w_uk; a.w_g = (const T*)L.w_uv; a.decay_rate = L.f_b; a.dt_bias = L.f_c;
    a.norm_w = L.f_a; a.state = (float*)kv->v[run]; a.R = hc.ring_len; a.eps = m->hyb->eps; a.out = (T*)b.mix;
    TRY(vn_delta_step(ctx, a));
    return VN_OK;
  }
  TRY(vn_delta_inputs(ctx, cv, in));
  if (rows.max_n > hc.pending)
    VN_LAUNCH(ctx, (conv_tail_kernel<T, Src, true>), dim3(ceil_div(cv.C, 256), rows.n_ent), 256, 0, cv, rows, hc.pending);
  GemmArgs g = gemm_args(b.low_a, L.rap, L.w_uk, H * d, L.rap, M, "gemm_delta_a2");
  g.C = b.g; g.ldc = H * d;
  TRY(linear(m, g));
  const long long ng = (long long)M * H * d;
  VN_LAUNCH(ctx, delta_decay_kernel, (unsigned)ceil_div(ng, 256ll), 256, 0, b.g, L.f_b, L.f_c, ng, H, d);
  g = gemm_args(b.low_g, L.rgp, L.w_uv, H * vd, L.rgp, M, "gemm_delta_g2");
  g.C = b.gg; g.ldc = H * vd;
  TRY(linear(m, g));
  DeltaRuleArgs a;
  a.q = b.dq; a.k = b.dk; a.v = b.dv; a.g = b.g; a.beta = b.beta; a.o = b.o; a.state = (float*)kv->v[run];
  a.R = hc.ring_len; a.H = H; a.KH = KH; a.d = d; a.vd = vd; a.rows = rows;
  TRY(vn_delta_scan(ctx, a));
  const long long nh = (long long)M * H;
  VN_LAUNCH(ctx, delta_out_kernel<T>, (unsigned)ceil_div(nh, 8ll), 256, 0, b.o, b.gg, L.f_a, (T*)b.mix, nh, vd, m->hyb->eps);
  return VN_OK;
}

// Grouped-query attention.  S: Src, or the 16-bit matrix of a forward of many rows
template <typename T, typename S>
int32_t attention(vn_model* m, const void* in_rows, vn_kv* kv, Cache& hc, const HLayer& L, int run, const Rows& rows, const Buffers& b) {
  vn_ctx* ctx = m->ctx;
  const Model& hm = *m->hyb;
  const int M = rows.M, D = hm.D, from = hm.runs[run].kv_run;
  ConvIn<T, S, false> cv;
  TRY(project(m, gemm_args(in_rows, D, L.w_in, L.n_in, D, M, "gemm_attn_in"), b.proj, &cv.src));
  cv.ring = (T*)hc.ring[run]; cv.RC = L.taps - 1 + hc.pending; cv.C = L.conv_ch(); cv.taps = L.taps; cv.w = L.conv; cv.named = L.conv_named;
  PagedAttnArgs a;
  a.H = L.H; a.KH = L.KH; a.d = L.d; a.vd = L.vd; a.P = L.P; a.window = L.window; a.chunk = L.chunk; a.scale = L.scale; a.softcap = L.softcap; a.rd = L.rd;
  a.interleaved = L.interleaved; a.qn = L.f_a; a.kn = L.f_b; a.eps = hm.eps;
  cv.bias = L.f_c;
  a.rope = L.rope >= 0 ? hm.ropes[L.rope].table : nullptr;
  a.own_kv = from == run;
  a.kplane = kv->k[from]; a.vplane = kv->v[from]; a.table = hc.table_dev; a.max_pages = hc.max_pages;
  a.col_g = L.gated ? L.conv_ch() : -1;
  a.gate_head = L.gated == GATE_HEAD;
  a.temp = L.temp;
  a.q = b.q; a.out = b.mix; a.pending = hc.pending; a.rows = rows;
  const bool mma = m->cfg.bf16 && attn_mma_ok(L.P) && !m->force_simt_attn;
  if constexpr (std::is_same<T, __nv_bfloat16>::value && std::is_same<S, Src>::value) {
    if (mma && rows.max_n == 1) {
      const int ctas = L.KH * ceil_div(L.H / L.KH, 16) * M;
      int keys = kv->max_seq;
      for (int reach : {L.window, L.chunk}) if (reach > 0) keys = std::min(keys, reach);
      a.splits = M > SPLIT_ROWS ? 1 : std::max(1, std::min(std::min(MAX_SPLITS, ceil_div(keys, 64)), 2 * ctx->sm_count / ctas));
      a.part_o = b.part_o; a.part_ml = b.part_ml;
      TRY(vn_tickets(ctx, &a.tickets));
      return vn_attn_step(ctx, cv, a);
    }
  }
  TRY(vn_attn_inputs(ctx, cv, a));
  if (rows.max_n > hc.pending && L.taps > 1)
    VN_LAUNCH(ctx, (conv_tail_kernel<T, S, false>), dim3(ceil_div(cv.C, 256), rows.n_ent), 256, 0, cv, rows, hc.pending);
  return vn_paged_attention<T, S>(ctx, cv.src, a, mma);
}

// Lightning attention; its output still has to be divided by the root mean square that b.ss [M, *n_ss] gives
template <typename T, typename S>
int32_t lightning(vn_model* m, const void* in_rows, vn_kv* kv, Cache& hc, const HLayer& L, int run, const Rows& rows, const Buffers& b, int* n_ss) {
  vn_ctx* ctx = m->ctx;
  Model& hm = *m->hyb;
  const int M = rows.M, D = hm.D, n_act = L.H * (2 * L.d + L.vd);
  const LightningPlan plan = vn_lightning_plan(ctx, m->cfg.bf16 != 0, L.H, L.d, L.vd, rows, hc.pending);
  LightningArgs a;
  a.H = L.H; a.d = L.d; a.vd = L.vd; a.decay = L.f_b; a.powers = L.f_c; a.norm_w = L.f_a; a.state = (float*)kv->v[run]; a.R = hc.ring_len;
  a.out = b.mix; a.ss = b.ss; a.n_ss = *n_ss = plan.n_ss; a.segments = plan.segments; a.seg_len = plan.seg_len; a.rows = rows;
  TRY(ensure_segments(m, plan.seg_bytes));
  a.seg_state = hm.seg;
  GemmArgs g = gemm_args(in_rows, D, L.w_in, L.n_in, D, M, "gemm_lightning_in");
  S s;
  if constexpr (std::is_same<S, Src>::value) {
    TRY(project(m, g, b.proj, &s));
    if constexpr (std::is_same<T, __nv_bfloat16>::value) {
      if (plan.chunked) {
        Mat<T> act;
        act.p = (const T*)b.lin; act.ld = L.n_in;
        const long long total4 = (long long)M * L.n_in / 4;
        if (n_act % 4 == 0)
          VN_LAUNCH(ctx, slices_act_kernel<T>, (unsigned)ceil_div(total4, 256ll), 256, 0, s, L.n_in, n_act, (int)POST_SILU, (T*)b.lin, L.n_in,
                    (float*)nullptr, total4);
        else
          VN_LAUNCH(ctx, slices_act1_kernel<T>, (unsigned)ceil_div(total4 * 4, 256ll), 256, 0, s, L.n_in, n_act, (int)POST_SILU, (T*)b.lin, total4 * 4);
        return vn_lightning_chunks(ctx, act, a);
      }
    }
    return vn_lightning_scan<T, S>(ctx, s, a);
  } else {
    g.post = POST_SILU; g.post_n = n_act;
    TRY(project(m, g, b.proj, &s));
    a.activated = 1;
    return plan.chunked ? vn_lightning_chunks(ctx, s, a) : vn_lightning_scan<T, S>(ctx, s, a);
  }
}

// ---- the forward ---------------------------------------------------------------------------------------------------
// where the output rows come from: all rows, the entries' last rows of a uniform batch, or a list (device)
struct Pick { const int* list = nullptr; int n = 0, mul = 1, add = 0; };

// final norm's rows in m->h -> logits
int32_t head(vn_model* m, int n_rows, float* out_logits) {
  const Model& hm = *m->hyb;
  GemmArgs g = gemm_args(m->h, hm.D, m->head, hm.vocab, hm.D, n_rows, "gemm_head");
  g.C = out_logits; g.ldc = hm.vocab;
  if (tc_rows(m, g)) {
    TcPlan direct;
    direct.error_flag = m->tc_error;
    return tc_launch(m->ctx, g, n_rows, direct);
  }
  return linear(m, g);
}

// out = glu(h W_gate^T, h W_up^T) of a gated feed-forward of padded width n, w: both matrices, rows in turn
template <typename T>
int32_t gated_up(vn_model* m, const void* w, int n, int act, float limit, int M, void* out, const char* tag) {
  vn_ctx* ctx = m->ctx;
  const int D = m->hyb->D;
  GemmArgs g = gemm_args(m->h, D, w, 2 * n, D, M, tag);
  if (tc_rows(m, g)) {
    int sp = 1;
    TRY(tc_partial(m, g, M, M, &sp));
    const long long pairs = (long long)M * n;
    VN_LAUNCH_PDL_BIT(ctx, 8, splitk_swiglu_kernel<T>, (unsigned)ceil_div(pairs, 512ll), 256, 0, m->partial, sp,
                      (long long)M * 2 * n, (T*)out, 2 * n, pairs, act, limit);
    return VN_OK;
  }
  g.C = out; g.ldc = n; g.epi = EPI_SWIGLU; g.act = act; g.act_limit = limit; g.c_bf16 = m->cfg.bf16;
  return linear(m, g);
}
template <typename T>
int32_t gated_up(vn_model* m, const HLayer& L, int M, const Buffers& b) {
  return gated_up<T>(m, L.w_gu, L.ffp, L.act, L.limit, M, b.act, "gemm_ff_gateup");
}

// act = PolyNorm(h W_up^T)
template <typename T, typename S>
int32_t poly_up(vn_model* m, const HLayer& L, int M, const Buffers& b) {
  vn_ctx* ctx = m->ctx;
  S z;
  TRY(project(m, gemm_args(m->h, m->hyb->D, L.w_gu, L.ffp, m->hyb->D, M, "gemm_ff_up"), b.proj, &z));
  const int n = L.ffp;
#define POLY(NV) VN_LAUNCH_PDL_LEVEL(ctx, 1, "poly_norm_kernel", (poly_norm_kernel<T, S, NV>), M, 256, 0, z, L.coef, (T*)b.act, L.ff, n, m->hyb->eps)
  if (n > 8192) POLY(0); else if (n <= 1024) POLY(1); else if (n <= 2048) POLY(2); else if (n <= 4096) POLY(4); else POLY(8);
#undef POLY
  return VN_OK;
}
template <typename T>
int32_t poly_up(vn_model* m, const HLayer& L, int M, const Buffers& b) {
  if constexpr (std::is_same<T, __nv_bfloat16>::value)
    if (M > 256) return poly_up<T, Mat<T>>(m, L, M, b);
  return poly_up<T, Src>(m, L, M, b);
}

// result of the expert that serves every row
template <typename T, typename S>
int32_t shared_expert(vn_model* m, const HLayer& L, int M, const Buffers& b, S* out) {
  TRY(gated_up<T>(m, L.w_sgu, L.sffp, L.act, L.s_limit, M, b.sact, "gemm_shared_gateup"));
  return project(m, gemm_args(b.sact, L.sffp, L.w_sdown, m->hyb->D, L.sffp, M, "gemm_shared_down"), b.sy, out, true);
}

// Mixture of experts: x += the weighted results of each row's experts and the gated one of the expert that serves every row (or
// their sum over its root mean square times the sublayer's norm); then as `next` says.  The rows are copied into expert order, times
// their weights where those belong to the input; few rows go as one segment per expert through split-K GEMMs, many as pieces of
// 256 rows.
template <typename T>
int32_t mixture(vn_model* m, const HLayer& L, int M, const Buffers& b, const Next& next) {
  vn_ctx* ctx = m->ctx;
  Model& hm = *m->hyb;
  const int D = hm.D, n = L.n_out() + L.joined(), S = L.slots(), F = L.ffp, mats = L.n_mats();
  const bool apart = L.sff && !L.joined();
  const bool bf = m->cfg.bf16;
  RouteIn r;
  TRY(project(m, gemm_args(m->h, D, L.w_router, L.n_router(), D, M, "gemm_router"), b.logits, &r.z));
  r.sigmoid = L.sigmoid; r.shared_gate = L.sff ? b.sgate : nullptr; r.shared_slot = L.joined();
  r.correction = L.correction; r.M = M; r.E = L.n_out(); r.top = L.top; r.groups = L.exp_groups; r.keep = L.keep;
  r.slot_expert = b.slot_expert; r.slot_w = b.slot_w; r.count = hm.exp_count;
  r.rows = route_rows(M);
  VN_LAUNCH_PDL_LEVEL(ctx, 1, "route_kernel", route_kernel, ceil_div(M, ROUTE_WARPS * r.rows), 32 * ROUTE_WARPS, route_smem(r.E, L.exp_groups), r);
  AddExperts<T, Src> few;          // results in split-K slices
  few.h = (const T*)m->h; few.slot_pos = b.slot_pos; few.slot_expert = b.slot_expert; few.slot_w = L.weigh_input ? nullptr : b.slot_w; few.top = S; few.n_real = mats; few.D = D;
  few.count = hm.exp_count; few.cursor = hm.exp_cur; few.n_count = n;
  few.y.ld = D;
  if (apart) few.shared_gate = r.shared_gate; else few.slot_gate = r.shared_gate;
  const float* scale = L.weigh_input ? b.slot_w : nullptr;
  GemmArgs up, down;
  up.A = b.hs; up.lda = D; up.W = L.w_gu; up.ldw = D; up.w_stride = (long long)2 * F * D; up.N = 2 * F; up.K = D; up.tag = "gemm_expert_gateup";
  up.C = b.act; up.ldc = F; up.epi = EPI_SWIGLU; up.act = L.act; up.act_limit = L.limit; up.c_bf16 = bf;
  down.A = b.act; down.lda = F; down.W = L.w_down; down.ldw = F; down.w_stride = (long long)D * F; down.N = D; down.K = F; down.tag = "gemm_expert_down";
  down.C = b.ey; down.ldc = D; down.c_bf16 = bf;
  up.M = down.M = M;
  const bool tc = bf && m->use_tc && D % 8 == 0 && tc_detail::encode_fn() != nullptr;
  if (tc && M <= 256) {
    if (apart) TRY((shared_expert<T, Src>(m, L, M, b, &few.shared)));
    VN_LAUNCH_PDL_LEVEL(ctx, 1, "mod_dispatch_kernel", mod_dispatch_kernel<T>, M * S, 128, 0, (const T*)m->h, b.slot_expert, hm.exp_count, hm.exp_off, hm.exp_cur,
                        b.slot_pos, (T*)b.hs, n, S, D, scale);
    up.seg_off = down.seg_off = hm.exp_off; up.seg_cnt = down.seg_cnt = hm.exp_count; up.nseg = down.nseg = mats;
    const int active = std::min(mats, M * S);          // segments with rows, at most
    int sp = 1;
    TRY(tc_partial(m, up, (long long)M * S, (long long)M * S, &sp, active));
    const long long pairs = (long long)M * S * F;
    VN_LAUNCH_PDL_BIT(ctx, 8, splitk_swiglu_kernel<T>, (unsigned)ceil_div(pairs, 512ll), 256, 0, m->partial, sp, (long long)M * S * 2 * F, (T*)b.act, 2 * F,
                      pairs, L.act, L.limit);
    TRY(tc_partial(m, down, (long long)M * S, (long long)M * S, &sp, active));
    few.y.p = m->partial; few.y.splits = sp; few.y.pstride = (long long)M * S * D;
    return close_rows<T>(m, few, M, L.post[1], next);
  }
  VN_LAUNCH(ctx, mod_offsets_kernel, 1, 32, 0, hm.exp_count, hm.exp_off, hm.exp_cur, n);
  VN_LAUNCH(ctx, mod_scatter_kernel, ceil_div(M * S, 256), 256, 0, b.slot_expert, hm.exp_off, hm.exp_cur, b.sorted_row, b.slot_pos, M * S, S, scale, scale ? b.sorted_w : (float*)nullptr);
  const float* sorted_w = scale ? b.sorted_w : nullptr;
  if (tc) {
    int *off = b.sub_seg, *cnt = off + b.sub_cap, *w = cnt + b.sub_cap;
    VN_LAUNCH(ctx, mod_subseg_kernel, 1, 32, 0, (const int*)hm.exp_count, (const int*)hm.exp_off, mats, off, cnt, w, b.sub_cap);
    VN_LAUNCH(ctx, gather_sorted_kernel<T>, M * S, 128, 0, (const T*)m->h, (const int*)b.sorted_row, (T*)b.hs, D, sorted_w);
    TRY(ensure_partial(m, 1024));
    for (GemmArgs* g : {&up, &down}) {
      g->M = 256; g->seg_off = off; g->seg_cnt = cnt; g->seg_w = w; g->n_w = mats; g->nseg = b.sub_cap;
      TcPlan plan;
      plan.error_flag = m->tc_error;
      TRY(launch_gemm_tc(ctx, *g, (long long)M * S, plan));
    }
  } else {                                                // the kernels of any shape gather rows themselves, as they are
    if (scale) {
      VN_LAUNCH(ctx, gather_sorted_kernel<T>, M * S, 128, 0, (const T*)m->h, (const int*)b.sorted_row, (T*)b.hs, D, sorted_w);
    } else {
      up.A = m->h; up.a_rows = b.sorted_row;
    }
    for (GemmArgs* g : {&up, &down}) {
      g->seg_off = hm.exp_off; g->seg_cnt = hm.exp_count; g->nseg = mats;
      TRY(linear(m, *g));
    }
  }
  if constexpr (std::is_same<T, __nv_bfloat16>::value) {
    AddExperts<T, Mat<T>> y;
    y.y.p = (const T*)b.ey; y.y.ld = D;
    y.h = few.h; y.slot_pos = few.slot_pos; y.slot_expert = few.slot_expert; y.slot_w = few.slot_w; y.shared_gate = few.shared_gate; y.slot_gate = few.slot_gate; y.top = S; y.n_real = few.n_real; y.D = D;
    y.count = few.count; y.cursor = few.cursor; y.n_count = n;
    if (apart) TRY((shared_expert<T, Mat<T>>(m, L, M, b, &y.shared)));
    return close_rows<T>(m, y, M, L.post[1], next);
  } else {
    few.y.p = (const float*)b.ey;
    if (apart) TRY((shared_expert<T, Src>(m, L, M, b, &few.shared)));
    return close_rows<T>(m, few, M, L.post[1], next);
  }
}

// x += norm(W_proj (gelu(W_gate x) * e)): e is the layer's part of the tokens' side embeddings, m->h holds x
template <typename T>
int32_t side_input(vn_model* m, const int64_t* tokens, const HLayer& L, int layer, int M, const Buffers& b, const Next& next) {
  vn_ctx* ctx = m->ctx;
  const Model& hm = *m->hyb;
  const int D = hm.D;
  Src gate;
  TRY(project(m, gemm_args(m->h, D, L.w_sgate, up4(hm.side), D, M, "gemm_side_gate"), b.proj, &gate));
  const long long total = (long long)M * hm.sidep;
  VN_LAUNCH_PDL_LEVEL(ctx, 1, "side_act_kernel", side_act_kernel<T>, (unsigned)ceil_div(total, 256ll), 256, 0, gate, (const long long*)tokens, hm.vocab,
                      (const T*)hm.side_embed, (long long)hm.layers.size() * hm.side, layer * hm.side, hm.side, (T*)b.side_act, hm.sidep, total);
  return close_normed<T>(m, gemm_args(b.side_act, hm.sidep, L.w_sproj, D, hm.sidep, M, "gemm_side_proj"), nullptr, b.proj, L.s_norm, next);
}

// act = relu(h W_up^T)^2, and the raw gate of the result beside it when the model has one
template <typename T>
int32_t plain_up(vn_model* m, const HLayer& L, int M, const Buffers& b, Src* gate) {
  vn_ctx* ctx = m->ctx;
  const Model& hm = *m->hyb;
  const int D = hm.D, n = L.ffp + (hm.res_gate ? D : 0);
  Src s;
  TRY(project(m, gemm_args(m->h, D, L.w_gu, n, D, M, "gemm_ff_up"), b.proj, &s));
  if (n % 4 == 0) {
    const long long total4 = (long long)M * n / 4;
    VN_LAUNCH_PDL_BIT(ctx, 8, slices_act_kernel<T>, (unsigned)ceil_div(total4, 256ll), 256, 0, s, n, L.ffp, (int)POST_RELU2, (T*)b.act,
                      L.ffp, hm.gate, total4);
    if (hm.res_gate) { *gate = Src(); gate->p = hm.gate; gate->ld = D; }
  } else {                                               // a plain matrix: the gate is read where it stands
    const long long total = (long long)M * L.ffp;
    VN_LAUNCH(ctx, slices_act1_kernel<T>, (unsigned)ceil_div(total, 256ll), 256, 0, s, L.ffp, L.ffp, (int)POST_RELU2, (T*)b.act, total);
    *gate = s;
    gate->p = s.p + L.ffp;
  }
  return VN_OK;
}
template <typename T>
int32_t plain_up(vn_model* m, const HLayer& L, int M, const Buffers& b, Mat<__nv_bfloat16>* gate) {
  const Model& hm = *m->hyb;
  GemmArgs g = gemm_args(m->h, hm.D, L.w_gu, L.ffp, hm.D, M, "gemm_ff_up");
  g.C = b.act; g.ldc = L.ffp; g.c_bf16 = 1; g.post = POST_RELU2; g.post_n = L.ffp;
  TRY(linear(m, g));
  return hm.res_gate ? project(m, gemm_args(m->h, hm.D, L.w_rg[1], hm.D, hm.D, M, "gemm_result_gate"), hm.gate, gate) : VN_OK;
}

// The forward over an arrangement of residual streams.  S: type of the projections' results
template <typename T, typename S>
int32_t forward_arranged(vn_model* m, vn_kv* kv, const int64_t* tokens, const Rows& rows, const Pick& pick, float* out_hidden,
                         float* out_logits) {
  vn_ctx* ctx = m->ctx;
  Model& hm = *m->hyb;
  Cache& hc = *kv->hyb;
  const int M = rows.M, D = hm.D, n_runs = (int)hm.runs.size();
  const bool single = rows.max_n == 1;
  struct Sub { int run, q; };
  std::vector<Sub> subs;
  for (int i = 0; i < n_runs; ++i) {
    subs.push_back({i, 0});
    if (hm.layers[hm.runs[i].layer].ff) subs.push_back({i, 1});
  }
  VN_LAUNCH(ctx, embed_pos_kernel<T>, M, 256, 0, (const long long*)tokens, (const T*)m->emb, hm.freq, m->x, hm.x0, rows, D,
            hm.vocab, m->status);
  StreamArgs<T, S> base;
  base.x = m->x; base.ns = std::max(1, hm.streams); base.D = D; base.layer_norm = hm.layer_norm; base.eps = hm.eps; base.rows = rows;
  // what a pass over the streams reads off for the next sublayer, or for the head when all rows go there in order
  const bool all_out = pick.n == M && !pick.list && pick.mul == 1 && pick.add == 0;
  auto next = [&](StreamArgs<T, S>& a, size_t k) {
    if (k < subs.size()) {
      const HLayer& L = hm.layers[hm.runs[subs[k].run].layer];
      const int q = subs[k].q;
      a.in = L.hc_in[q]; a.norm_w = q ? L.norm2 : L.norm1; a.h = (T*)m->h;
      if (!q && hm.in_taps && single) {
        a.hc = (T*)hm.hc; a.ring = (T*)hc.in_ring[subs[k].run]; a.conv_w = L.in_conv; a.taps = hm.in_taps;
        a.RC = hm.in_taps - 1 + hc.pending;
      }
    } else if (all_out) {
      a.norm_w = m->norm_f; a.h = (T*)m->h; a.h32 = out_hidden;
    }
  };
  {
    StreamArgs<T, S> a = base;
    a.first = hm.x0;
    next(a, 0);
    TRY(vn_streams(ctx, a, M));
  }
  for (size_t k = 0; k < subs.size(); ++k) {
    const int i = subs[k].run, q = subs[k].q;
    const HLayer& L = hm.layers[hm.runs[i].layer];
    Arena A;
    Buffers b;
    A.base = hm.ws;
    layout(hm, L, M, m->esz, A, b);
    StreamArgs<T, S> a = base;
    if (k == 0) a.first = hm.x0;
    if (hm.res_gate && !(q && L.ff_plain))
      TRY(project(m, gemm_args(m->h, D, L.w_rg[q], D, D, M, "gemm_result_gate"), hm.gate, &a.gate, true));
    GemmArgs out;
    if (!q) {
      const void* in_rows = m->h;
      if (hm.in_taps) {
        in_rows = hm.hc;
        if (!single) {
          ConvIn<T, Mat<T>, false> cv;
          cv.src.p = (const T*)m->h; cv.src.ld = D; cv.ring = (T*)hc.in_ring[i]; cv.RC = hm.in_taps - 1 + hc.pending; cv.C = D;
          cv.taps = hm.in_taps; cv.w = L.in_conv;
          TRY(vn_input_conv(ctx, cv, rows, hc.pending, (T*)hm.hc));
          if (rows.max_n > hc.pending && hm.in_taps > 1)
            VN_LAUNCH(ctx, (conv_tail_kernel<T, Mat<T>, false>), dim3(ceil_div(D, 256), rows.n_ent), 256, 0, cv, rows, hc.pending);
        }
      }
      if (L.kind == LATENT) TRY((latent_attention<T, Src>(m, in_rows, kv, hc, L, i, rows, b)));
      else if (L.kind == MAMBA1) TRY(mamba1<T>(m, in_rows, kv, hc, L, i, rows, b));
      else if (L.kind == DELTA) TRY(channel_delta<T>(m, in_rows, kv, hc, L, i, rows, b));
      else if (L.kind == ATTENTION) TRY((attention<T, S>(m, in_rows, kv, hc, L, i, rows, b)));
      else {
        TRY((lightning<T, S>(m, in_rows, kv, hc, L, i, rows, b, &a.n_ss)));
        a.ss = b.ss; a.ss_count = (float)(L.H * L.vd);
      }
      const int width = L.kind == MAMBA1 ? L.inner : L.H * L.vd;
      out = gemm_args(b.mix, width, L.w_o, D, width, M, "gemm_mix_out");
    } else {
      if (L.ff_plain) TRY(plain_up<T>(m, L, M, b, &a.gate)); else TRY(gated_up<T>(m, L, M, b));
      out = gemm_args(b.act, L.ffp, L.w_down, D, L.ffp, M, "gemm_ff_down");
    }
    TRY(project(m, out, hm.y, &a.y));
    a.gate_b = L.rg_b[q]; a.mix = L.hc_mix[q]; a.out = L.hc_out[q];
    next(a, k + 1);
    TRY(vn_streams(ctx, a, M));
    if (hm.probe && (k + 1 == subs.size() || subs[k + 1].run != i)) TRY(vn_streams_sum(ctx, m->x, hm.probe + (size_t)i * M * D, M, base.ns, D));
  }
  if (pick.n == 0) return VN_OK;
  if (!all_out) {
    StreamArgs<T, S> a = base;
    a.pick = pick.list; a.mul = pick.mul; a.add = pick.add; a.norm_w = m->norm_f; a.h = (T*)m->h; a.h32 = out_hidden;
    TRY(vn_streams(ctx, a, pick.n));
  }
  return out_logits ? head(m, pick.n, out_logits) : VN_OK;
}

// mixers that read the projection of many rows in 16 bits
template <typename T>
int32_t dense_projection_mixer(vn_model* m, const void* in_rows, vn_kv* kv, Cache& hc, const HLayer& L, int run, const Rows& rows, const Buffers& b) {
  auto run_as = [&](auto tag) -> int32_t {
    using S = decltype(tag);
    if (L.kind == LATENT) return latent_attention<T, S>(m, in_rows, kv, hc, L, run, rows, b);
    if (L.kind == MAMBA2) return mamba2<T, S>(m, in_rows, kv, hc, L, run, rows, b);
    return attention<T, S>(m, in_rows, kv, hc, L, run, rows, b);
  };
  if constexpr (std::is_same<T, __nv_bfloat16>::value)
    if (rows.M > 256) return run_as(Mat<T>());
  return run_as(Src());
}

template <typename T>
int32_t forward(vn_model* m, vn_kv* kv, const int64_t* tokens, const Rows& rows, const Pick& pick, float* out_hidden,
                float* out_logits) {
  vn_ctx* ctx = m->ctx;
  Model& hm = *m->hyb;
  Cache& hc = *kv->hyb;
  const int M = rows.M, D = hm.D, n_runs = (int)hm.runs.size();
  TRY(ensure_partial(m, 1024));
  if (hm.arranged) {
    if constexpr (std::is_same<T, __nv_bfloat16>::value)
      if (M > 256) return forward_arranged<T, Mat<T>>(m, kv, tokens, rows, pick, out_hidden, out_logits);
    return forward_arranged<T, Src>(m, kv, tokens, rows, pick, out_hidden, out_logits);
  }
  VN_LAUNCH(ctx, embed_pos_kernel<T>, M, 256, 0, (const long long*)tokens, (const T*)m->emb, hm.freq, m->x, hm.x0, rows, D,
            hm.vocab, m->status);
  auto enters_pass = [&](int i) { return i < n_runs && hm.runs[i].pass >= 0 && hm.runs[i].layer == hm.loop_start; };
  auto pass_entry = [&](int i) {
    PassEntry p;
    if (enters_pass(i) && hm.loop_add) { p.step = hm.loop_step + (long long)hm.runs[i].pass * D; p.x0 = hm.runs[i].pass > 0 ? hm.x0 : nullptr; }
    return p;
  };
  for (int i = 0; i < n_runs; ++i) {
    const HLayer& L = hm.layers[hm.runs[i].layer];
    Arena A;
    Buffers b;
    A.base = hm.ws;
    layout(hm, L, M, m->esz, A, b);
    if (enters_pass(i) && !hm.loop_add) {
      // x = W [x | x0] + step vector of the pass, and the first layer's norm
      VN_LAUNCH(ctx, concat_cast_kernel<T>, M, 256, 0, m->x, hm.x0, (T*)hm.cat, D);
      Src s;
      TRY(project(m, gemm_args(hm.cat, 2 * D, hm.w_loop, D, 2 * D, M, "gemm_loop_in"), b.proj, &s));
      VN_LAUNCH(ctx, rowsum_norm_kernel<T>, M, 256, 0, s, hm.loop_step + (long long)hm.runs[i].pass * D, 0, m->x, L.norm1,
                (T*)m->h, D, hm.eps);
    } else if (enters_pass(i) && (i == 0 || hm.probe)) {
      VN_LAUNCH(ctx, enter_pass_kernel<T>, M, 256, 0, pass_entry(i), m->x, L.norm1, (T*)m->h, D, hm.eps);
    } else if (i == 0) {
      VN_LAUNCH(ctx, rmsnorm_kernel<T>, M, 256, 0, m->x, L.norm1, (T*)m->h, (float*)nullptr, 1, 0, D, hm.eps);
    }
    Next next_layer;                                      // an entry that adds is part of the sublayer's end before it
    if (i + 1 < n_runs && (!enters_pass(i + 1) || (hm.loop_add && !hm.probe)))
      next_layer = {hm.layers[hm.runs[i + 1].layer].norm1, false, pass_entry(i + 1)};
    const Next after_ff = hm.side ? Next{nullptr, true, {}} : next_layer, after_mix = L.ff ? Next{L.norm2, false, {}} : after_ff;
    auto close = [&](const GemmArgs& g, const float* bias, const float* own_norm, const Next& next) {
      return own_norm ? close_normed<T>(m, g, bias, b.proj, own_norm, next) : close_block<T>(m, g, bias, next);
    };
    if (L.kind == MAMBA1) TRY(mamba1<T>(m, m->h, kv, hc, L, i, rows, b));
    else if (L.kind == DELTA) TRY(channel_delta<T>(m, m->h, kv, hc, L, i, rows, b));
    else TRY((dense_projection_mixer<T>(m, m->h, kv, hc, L, i, rows, b)));
    const int width = L.kind == MAMBA1 ? L.inner : L.H * L.vd;
    TRY(close(gemm_args(b.mix, width, L.w_o, D, width, M, "gemm_mix_out"), L.o_b, L.post[0], after_mix));
    if (L.n_exp) {
      TRY(mixture<T>(m, L, M, b, after_ff));
    } else if (L.ff) {
      if (L.poly) TRY(poly_up<T>(m, L, M, b)); else TRY(gated_up<T>(m, L, M, b));
      TRY(close(gemm_args(b.act, L.ffp, L.w_down, D, L.ffp, M, "gemm_ff_down"), nullptr, L.post[1], after_ff));
    }
    if (hm.side) TRY(side_input<T>(m, tokens, L, hm.runs[i].layer, M, b, next_layer));
    if (hm.probe)
      VN_CUDA(ctx, cudaMemcpyAsync(hm.probe + (size_t)i * M * D, m->x, (size_t)M * D * 4, cudaMemcpyDeviceToDevice, ctx->stream));
  }
  if (pick.n == 0) return VN_OK;
  if (pick.list)
    VN_LAUNCH(ctx, rmsnorm_pick_kernel<T>, pick.n, 256, 0, m->x, m->norm_f, (T*)m->h, out_hidden, pick.list, 1, 0, D, hm.eps);
  else
    VN_LAUNCH(ctx, rmsnorm_kernel<T>, pick.n, 256, 0, m->x, m->norm_f, (T*)m->h, out_hidden, pick.mul, pick.add, D, hm.eps);
  return out_logits ? head(m, pick.n, out_logits) : VN_OK;
}

// ---- cache -----------------------------------------------------------------------------------------------------------
int32_t push_table(vn_ctx* ctx, Cache& hc, int slot) {
  VN_CUDA(ctx, cudaMemcpyAsync(hc.table_dev + (size_t)slot * hc.max_pages, hc.table.data() + (size_t)slot * hc.max_pages,
                               (size_t)hc.max_pages * 4, cudaMemcpyHostToDevice, ctx->stream));
  return VN_OK;
}

// rotation tables for at least `rows` positions
int32_t ensure_ropes(vn_model* m, int rows) {
  vn_ctx* ctx = m->ctx;
  for (Rope& r : m->hyb->ropes) {
    if (r.rows >= rows || r.freq.empty()) continue;
    const int n = std::max(rows, 2 * r.rows), pairs = (int)r.freq.size();
    float2* t = nullptr;
    double* f = nullptr;
    TRY(dev_alloc(ctx, (void**)&t, (size_t)n * pairs * sizeof(float2)));
    TRY(dev_alloc(ctx, (void**)&f, (size_t)pairs * 8));
    VN_CUDA(ctx, cudaMemcpyAsync(f, r.freq.data(), (size_t)pairs * 8, cudaMemcpyHostToDevice, ctx->stream));
    const int32_t st = vn_rope_table(ctx, f, pairs, r.amp, n, t);
    VN_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
    cudaFree(f);
    if (r.table) m->hyb->retired.push_back(r.table);
    r.table = t; r.rows = n;
    TRY(st);
  }
  return VN_OK;
}

int32_t cache_create(vn_model* m, vn_kv* kv, int pool_tokens, int pending) {
  vn_ctx* ctx = m->ctx;
  Model& hm = *m->hyb;
  Cache* hc = kv->hyb = new Cache();
  hc->pending = pending;
  hc->ring_len = pending + 1;
  hc->slots = kv->max_batch;
  hc->max_pages = ceil_div(kv->max_seq, KV_PAGE);
  hc->pooled = pool_tokens > 0;
  hc->n_pages = hc->pooled ? ceil_div(pool_tokens, KV_PAGE) : hc->slots * hc->max_pages;
  hc->table.assign((size_t)hc->slots * hc->max_pages, 0);
  hc->used.assign(hc->slots, 0);
  if (hc->pooled) {
    for (int p = hc->n_pages - 1; p >= 0; --p) hc->free_pages.push_back(p);
  } else {
    for (size_t i = 0; i < hc->table.size(); ++i) hc->table[i] = (int)i;
    hc->used.assign(hc->slots, hc->max_pages);
  }
  TRY(dev_alloc(ctx, (void**)&hc->table_dev, hc->table.size() * 4));
  VN_CUDA(ctx, cudaMemcpyAsync(hc->table_dev, hc->table.data(), hc->table.size() * 4, cudaMemcpyHostToDevice, ctx->stream));
  TRY(ensure_ropes(m, kv->max_seq));
  for (size_t i = 0; i < hm.runs.size(); ++i) {
    const Run& r = hm.runs[i];
    const HLayer& L = hm.layers[r.layer];
    void *a = nullptr, *b = nullptr, *c = nullptr, *in = nullptr;
    int32_t st = VN_OK;
    if (hm.in_taps) st = dev_alloc(ctx, &in, (size_t)hc->slots * (hm.in_taps - 1 + pending) * hm.D * m->esz);
    hc->in_ring.push_back(in);
    if (st == VN_OK && L.kind == ATTENTION) st = dev_alloc(ctx, &c, (size_t)hc->slots * (L.taps - 1 + pending) * L.conv_ch() * m->esz);
    hc->ring.push_back(c);
    if (st != VN_OK) return st;
    if (L.kind == ATTENTION) {
      const size_t plane = (size_t)hc->n_pages * KV_PAGE * L.KH * L.P * m->esz;
      if (r.kv_run == (int)i) st = dev_alloc(ctx, &a, plane);
      if (st == VN_OK && a) st = dev_alloc(ctx, &b, plane);
    } else if (L.kind == LIGHTNING) {
      st = dev_alloc(ctx, &b, (size_t)hc->slots * hc->ring_len * L.state_elems() * 4);
    } else if (L.kind == LATENT) {
      st = dev_alloc(ctx, &a, (size_t)hc->n_pages * KV_PAGE * L.Rp * m->esz);
    } else {
      st = dev_alloc(ctx, &a, (size_t)hc->slots * (L.taps - 1 + pending) * L.conv_ch() * m->esz);
      if (st == VN_OK) st = dev_alloc(ctx, &b, (size_t)hc->slots * hc->ring_len * L.state_elems() * 4);
    }
    kv->k.push_back(a); kv->v.push_back(b);
    TRY(st);
  }
  VN_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
  return VN_OK;
}

void cache_free(vn_kv* kv) {
  if (!kv->hyb || kv->parent) return;
  if (kv->hyb->table_dev) cudaFree(kv->hyb->table_dev);
  for (void* p : kv->hyb->ring) if (p) cudaFree(p);
  for (void* p : kv->hyb->in_ring) if (p) cudaFree(p);
  delete kv->hyb;
  kv->hyb = nullptr;
}

// pages for `tokens` positions of a slot (pooled caches); *grew tells whether the device table is behind
int32_t reserve(vn_ctx* ctx, Cache& hc, int slot, int tokens) {
  const int need = ceil_div(tokens, KV_PAGE);
  if (!hc.pooled || need <= hc.used[slot]) return VN_OK;
  if (need - hc.used[slot] > (int)hc.free_pages.size())
    return vn_fail(ctx, VN_ERR_OVERFLOW, "KV cache overflow: sequence %d needs %d more pages of %d tokens, the pool has %zu free",
                   slot, need - hc.used[slot], KV_PAGE, hc.free_pages.size());
  while (hc.used[slot] < need) {
    hc.table[(size_t)slot * hc.max_pages + hc.used[slot]++] = hc.free_pages.back();
    hc.free_pages.pop_back();
  }
  return push_table(ctx, hc, slot);
}

// a slot whose sequence is gone gives its pages back (later work of the stream may overwrite them)
void release(Cache& hc, int slot) {
  if (!hc.pooled) return;
  while (hc.used[slot] > 0) hc.free_pages.push_back(hc.table[(size_t)slot * hc.max_pages + --hc.used[slot]]);
}

int32_t run_forward(vn_model* m, vn_kv* kv, const int64_t* tokens, const Rows& rows, const Pick& pick, float* hidden, float* logits) {
  TRY(ensure(m, rows.M));
  if (m->cfg.bf16) return forward<__nv_bfloat16>(m, kv, tokens, rows, pick, hidden, logits);
  return forward<float>(m, kv, tokens, rows, pick, hidden, logits);
}

// T new rows for sequences 0 .. B-1 of `kv` (a cache or a view); capacity has been checked
int32_t forward_uniform(vn_model* m, vn_kv* kv, const int64_t* tokens, int B, int T, int slot_offset, float* hidden,
                        float* logits, int last_only) {
  vn_ctx* ctx = m->ctx;
  Cache& hc = *kv->hyb;
  VN_REQUIRE(ctx, slot_offset == 0 || slot_offset + T <= hc.pending,
             "%d uncommitted rows, +%d: this cache keeps %d (max_pending)", slot_offset, T, hc.pending);
  if (hc.pooled) {
    // the host's bound on a length may be above it after cut-back appends: exact before a page is taken
    bool grow = false;
    for (int b = 0; b < B; ++b) grow |= ceil_div(kv_ub(kv, b) + slot_offset + T, KV_PAGE) > hc.used[kv->parent_first + b];
    if (grow) { std::vector<int32_t> lens(kv->max_batch); TRY(vn_kv_lengths(kv, lens.data())); }
    for (int b = 0; b < B; ++b) TRY(reserve(ctx, hc, kv->parent_first + b, kv_ub(kv, b) + slot_offset + T));
  }
  Rows r;
  r.T = T; r.slot0 = kv->parent_first; r.off = slot_offset; r.n_ent = B; r.M = B * T; r.max_n = T;
  r.lens = kv->lens - kv->parent_first;
  Pick p;
  if (last_only) { p.n = B; p.mul = T; p.add = T - 1; } else { p.n = B * T; }
  return run_forward(m, kv, tokens, r, p, hidden, logits);
}

// a ragged batch: entry e brings counts[e] rows for sequence slots[e]; everything it appends is committed
int32_t forward_ragged(vn_model* m, vn_kv* kv, const int64_t* tokens, int n_ent, const int* slots, const int* counts, int n_out,
                       const int* out_rows, float* hidden, float* logits) {
  vn_ctx* ctx = m->ctx;
  Cache& hc = *kv->hyb;
  Model& hm = *m->hyb;
  int M = 0, max_n = 0;
  std::vector<char> seen(kv->max_batch, 0);
  for (int e = 0; e < n_ent; ++e) {
    if (slots[e] < 0 || slots[e] >= kv->max_batch) return vn_fail(ctx, VN_ERR_INDEX, "sequence %d out of range (%d)", slots[e], kv->max_batch);
    VN_REQUIRE(ctx, counts[e] >= 1 && !seen[slots[e]], "entry %d: no rows, or sequence %d named twice", e, slots[e]);
    seen[slots[e]] = 1;
    M += counts[e];
    max_n = std::max(max_n, counts[e]);
  }
  bool exact = false;
  for (int e = 0; e < n_ent; ++e) {
    if (kv_ub(kv, slots[e]) + counts[e] > kv->max_seq && !exact) {
      std::vector<int32_t> lens(kv->max_batch);
      TRY(vn_kv_lengths(kv, lens.data()));
      exact = true;
    }
    if (kv_ub(kv, slots[e]) + counts[e] > kv->max_seq)
      return vn_fail(ctx, VN_ERR_OVERFLOW, "KV cache overflow: sequence %d holds %d, +%d exceeds the capacity %d", slots[e],
                     kv_ub(kv, slots[e]), counts[e], kv->max_seq);
  }
  for (int i = 0; i < n_out; ++i) VN_REQUIRE(ctx, out_rows[i] >= 0 && out_rows[i] < M, "output row %d of %d", out_rows[i], M);
  for (int e = 0; e < n_ent; ++e)
    TRY(reserve(ctx, hc, kv->parent_first + slots[e], kv_ub(kv, slots[e]) + counts[e]));
  // tables: slot, first row, rows of the entries; entry of each row; wanted rows
  std::vector<int> t((size_t)3 * n_ent + M + n_out);
  int *ts = t.data(), *tr = ts + n_ent, *tc = tr + n_ent, *te = tc + n_ent, *to = te + M;
  for (int e = 0, r = 0; e < n_ent; ++e) {
    ts[e] = kv->parent_first + slots[e]; tr[e] = r; tc[e] = counts[e];
    for (int i = 0; i < counts[e]; ++i) te[r++] = e;
  }
  std::copy(out_rows, out_rows + n_out, to);
  if ((int)t.size() > hm.meta_cap) {
    VN_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
    if (hm.meta) cudaFree(hm.meta);
    hm.meta = nullptr; hm.meta_cap = 0;
    TRY(dev_alloc(ctx, (void**)&hm.meta, t.size() * 2 * 4));
    hm.meta_cap = (int)t.size() * 2;
  }
  VN_CUDA(ctx, cudaMemcpyAsync(hm.meta, t.data(), t.size() * 4, cudaMemcpyHostToDevice, ctx->stream));
  Rows r;
  r.n_ent = n_ent; r.M = M; r.max_n = max_n;
  r.slot = hm.meta; r.row0 = r.slot + n_ent; r.cnt = r.row0 + n_ent; r.ent = r.cnt + n_ent;
  r.lens = kv->lens - kv->parent_first;
  Pick p;
  p.list = r.ent + M; p.n = n_out;
  TRY(run_forward(m, kv, tokens, r, p, hidden, logits));
  VN_LAUNCH(ctx, rows_advance_kernel, ceil_div(n_ent, 128), 128, 0, r, kv->lens - kv->parent_first);
  for (int e = 0; e < n_ent; ++e) kv_ub(kv, slots[e]) += counts[e];
  return VN_OK;
}

}  // namespace hybrid
