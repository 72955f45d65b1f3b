// Dabodra: a decoder-only design on one fp32 residual that norms what a sublayer gives and not what it reads, whose mixers
// are sliding-window attention on values that are the projected keys, or the gated delta rule, and whose feed-forward is a
// mixture of group-limited, sigmoid-scored experts beside a shared expert.
//
//   x[t]     = N_e(embed[token]),  N(u) = u / sqrt(mean(u^2) + eps) * (1 + w)                            (hyper.cu embed_normed)
//   sublayer : x <- x + N(f(x)); f reads x itself                                                        (hyper.cu sandwich_step)
//   attention: q = W_q h, k = W_k h, v = k; q and k RMS-normed as whole rows with weights, then the first rot.dims dimensions
//              of every head rotated in pairs (2i, 2i + 1); grouped heads; score = scale q.k over the keys j with
//              0 <= i - j < mask.size; softmax with exp(sink_h) in its denominator; W_o  (window_attention.cu: conv_qk_prep without
//              a convolution, window_attention)
//   delta    : q, k, v through a short causal convolution and SiLU, q and k of every head made unit vectors (q times
//              dim^(-1/2)); beta = sigmoid(W_b h), g = exp(-exp(A_log) softplus(W_a h + dt_bias)) per head;
//              S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q; o / rms(o) * w * silu(W_g h) per head; W_o
//                                                                        (ssm.cu, delta.cu, gla.cu recurrent_out_gate)
//   ff       : s = sigmoid(W_r h) in fp32; the `top` largest s + correction among the `keep` groups whose two largest s + correction
//              have the largest sum; weights scale * s / (sum of the chosen s + 1e-20); expert(h) = W_down (silu(W_gate h) * W_up h);
//              plus the shared expert                                                                     (moe.cu, linear.cu)
//   logits   = head N_f(x)
//
// Per layer the kernel sequence is: the residual boundary (previous output's norm and addition, the rounded row the next
// sublayer reads), ONE input projection for everything that reads the mixer's input, the mixer's own kernels, its output
// projection, the boundary, and the feed-forward.  Every size and constant comes from config.json; matrices and activations
// are bf16 or fp32; the residual, norms, softmax, router, gates and unit norms of the recurrence and its state are fp32 either
// way.  A sequence's state slot holds the carried convolution inputs and the matrices of every delta layer; the page pool
// holds keys and values of every attention layer, and pages behind every window go back to it while a sequence runs.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <string.h>

#include <algorithm>

#include "errors.h"
#include "gemm.h"
#include "model.h"

namespace b200 {
namespace {

typedef __nv_bfloat16 bf16;

constexpr float kUnitEps = 1e-6f;      // inside the root of the delta rule's unit norms
constexpr float kWeightSumEps = 1e-20f;   // added to the sum of the chosen experts' scores

enum MixerKind { MIX_ATTENTION = 0, MIX_DELTA = 1 };

struct LayerSpec {
  int kind = MIX_ATTENTION;
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
  // attention
  int window = 1 << 30, rot_dims = 0;
  double rot_base = 10000.0;
  float scale = 1.f;
  // delta
  int taps = 0;                            // 0 until the config or the checkpoint says it
  // feed-forward
  bool mlp = false, shared = false;
  int experts = 0, top = 0, groups = 1, keep = 1, ff = 0, sff = 0;
  float route_scale = 1.f;
  // column layout of the input projection's output row: [q | k] (attention), [q | k | v] (delta) are one run of columns
  int n_in = 0, off_qkv = 0, off_g = 0, off_b = 0, off_a = 0;
  int k_out = 0, n_sh = 0, conv_c = 0;
  size_t conv_floats = 0, rec_floats = 0;  // the layer's part of a state slot: carried convolution inputs, recurrent state
};

struct LayerWeights {
  void* w_in = nullptr;     // [n_in, width]
  void* w_out = nullptr;    // [width, k_out]
  float *norm1 = nullptr, *norm2 = nullptr;                    // 1 + stored weight
  float *q_norm = nullptr, *k_norm = nullptr, *sink = nullptr; // attention: [heads * dim], [kv_heads * dim], [heads]
  float2* rope = nullptr;   // attention: [max_model_len][rot_dims / 2]
  float *conv_w = nullptr, *dt_b = nullptr, *rate = nullptr, *o_norm = nullptr;   // delta: [conv_c, taps], [heads], [heads] (-exp(A_log)), [vdim]
  void* router = nullptr;   // [experts, width]
  float* correction = nullptr;
  void* e_gu = nullptr;     // [experts][2 ff][width]  gate rows, then up rows (or in turns, see il_e)
  void* e_down = nullptr;   // [experts][width][ff]
  void* sh_in = nullptr;    // [n_sh, width]: gate [sff] | up [sff] (or in turns, see il_s)
  void* sh_down = nullptr;  // [width, sff]
  GemmPlan p_in, p_out, p_shin, p_shdown;
  GroupedPlan g_egu, g_edown;
  CUtensorMap xg_h, xg_act;                                    // the grouped form's views of the sorted rows and of the hidden rows
  CUtensorMap xm_out[kGemmNumBlockN], xm_shact[kGemmNumBlockN];
  bool tc_in = false, tc_out = false, tc_shin = false, tc_shdown = false, tc_experts = false;
  // gate and up rows in alternating blocks of 64, so that one GEMM tile holds both and its epilogue can join them
  bool il_e = false, il_s = false;
};

struct LayerRun {
  void* cache = nullptr;    // attention: [num_blocks * page][kv_heads * dim (keys) | kv_heads * dim (values)]
  float* conv = nullptr;    // delta: [slots][taps - 1][channels]
  float* state = nullptr;   // delta: [slots][heads][dim][vdim]
};

bool jnum(const JVal* o, const char* k, double* out) {
  const JVal* v = o ? o->get(k) : nullptr;
  if (!v || v->type != JVal::Num) return false;
  *out = v->num;
  return true;
}

class Dabodra : public Model {
 public:
  DType dt;
  int V = 0, W = 0;
  float eps = 1e-5f;
  std::vector<LayerSpec> spec;
  std::vector<LayerWeights> wts;
  std::vector<LayerRun> run;
  ModelEnv env;
  void *embed = nullptr, *head = nullptr;
  float *emb_w = nullptr, *fin_w = nullptr;
  // activations
  float *x = nullptr, *qn = nullptr, *o32 = nullptr, *logits = nullptr, *scores = nullptr, *topw = nullptr, *edown = nullptr;
  void *h = nullptr, *inb = nullptr, *xc = nullptr, *yb = nullptr, *ao = nullptr, *fo = nullptr, *hrow = nullptr;
  void *egu = nullptr, *eact = nullptr, *sh = nullptr, *shact = nullptr, *sdown = nullptr, *hsorted = nullptr, *edown16 = nullptr;
  int *topi = nullptr, *sorted_rows = nullptr, *tile_group = nullptr, *pair_pos = nullptr, *iota = nullptr;
  int* expert_rows = nullptr;
  int* kernel_error = nullptr;   // pinned: a kernel whose wait ran out leaves a mark here
  int row_cap = 0, moe_cap = 0;
  std::vector<void*> allocs;
  float* gemm_ws = nullptr;
  int* gemm_counters = nullptr;
  int few_rows = 16;
  bool whole = true;
  CUtensorMap xm_h[kGemmNumBlockN];
  bool use_tc = false;

  explicit Dabodra(DType d) : dt(d) {}
  ~Dabodra() override {
    for (auto& w : wts) {
      if (w.tc_in) gemm_plan_destroy(&w.p_in);
      if (w.tc_out) gemm_plan_destroy(&w.p_out);
      if (w.tc_shin) gemm_plan_destroy(&w.p_shin);
      if (w.tc_shdown) gemm_plan_destroy(&w.p_shdown);
    }
    if (pe0) { cudaEventDestroy(pe0); cudaEventDestroy(pe1); }
    if (kernel_error) cudaFreeHost(kernel_error);
    for (void* p : allocs) cudaFree(p);
  }
  const char* arch() const override { return "Dabodra"; }
  int vocab() const override { return V; }

  size_t cache_bytes_per_block(int page) const override {
    size_t b = 0;
    for (auto& s : spec)
      if (s.kind == MIX_ATTENTION) b += static_cast<size_t>(page) * s.kv_heads * 2 * s.dim * dtype_bytes(dt);
    return b;
  }
  size_t state_bytes_per_slot() const override {
    size_t b = 0;
    for (auto& s : spec) b += (s.conv_floats + s.rec_floats) * sizeof(float);
    return b;
  }
  int cache_window() const override {
    int w = 0;
    for (auto& s : spec)
      if (s.kind == MIX_ATTENTION) {
        if (s.window >= 1 << 30) return 0;
        w = std::max(w, s.window);
      }
    return w;
  }

  // ------------------------------------------------------------ config.json
  bool parse(const JVal& c, std::string* err) {
    double d = 0;
    auto whole = [&](const JVal* o, const char* k, int lo, int* out, const std::string& where) {
      double v = 0;
      if (!jnum(o, k, &v) || v < lo || v != floor(v) || v > 2147483647.0) { *err = "config: " + where + k; return false; }
      *out = static_cast<int>(v);
      return true;
    };
    auto given = [](const JVal* o, const char* k) { const JVal* v = o ? o->get(k) : nullptr; return v && !v->is_null(); };
    if (!whole(&c, "vocab", 1, &V, "") || !whole(&c, "width", 1, &W, "")) return false;
    if (W > 12288) { *err = "config: width above 12288"; return false; }
    if (jnum(c.get("norm"), "eps", &d)) eps = static_cast<float>(d);
    const JVal* ls = c.get("layers");
    if (!ls || ls->type != JVal::Arr || ls->arr.empty()) { *err = "config: layers"; return false; }
    for (size_t i = 0; i < ls->arr.size(); ++i) {
      const JVal& L = ls->arr[i];
      const std::string where = "layer " + std::to_string(i) + " ", mw = where + "mixer.", rw = where + "mlp.router.";
      LayerSpec s;
      const JVal* ty = L.get("type");
      const JVal* mx = L.get("mixer");
      if (!ty || ty->type != JVal::Str) { *err = "config: " + where + "type"; return false; }
      if (!mx || mx->type != JVal::Obj) { *err = "config: " + where + "mixer"; return false; }
      if (!whole(mx, "heads", 1, &s.heads, mw) || !whole(mx, "dim", 1, &s.dim, mw)) return false;
      s.kv_heads = s.heads;
      s.vdim = s.dim;
      if (given(mx, "kv_heads") && !whole(mx, "kv_heads", 1, &s.kv_heads, mw)) return false;
      if (given(mx, "vdim") && !whole(mx, "vdim", 1, &s.vdim, mw)) return false;
      if (s.heads % s.kv_heads) { *err = "config: " + mw + "heads is no multiple of kv_heads"; return false; }
      if (ty->str == "attention") {
        s.kind = MIX_ATTENTION;
        if (s.vdim != s.dim) { *err = "config: " + mw + "vdim differs from dim (the values are the keys)"; return false; }
        if (s.dim > 256) { *err = "config: " + mw + "dim above 256"; return false; }
        if (given(mx, "mask") && given(mx->get("mask"), "size") && !whole(mx->get("mask"), "size", 1, &s.window, mw + "mask.")) return false;
        s.rot_dims = s.dim / 2 * 2;
        if (const JVal* rot = mx->get("rot")) {
          if (rot->is_null()) s.rot_dims = 0;
          if (given(rot, "dims") && !whole(rot, "dims", 0, &s.rot_dims, mw + "rot.")) return false;
          if (jnum(rot, "base", &d)) s.rot_base = d;
        }
        if (s.rot_dims > s.dim || s.rot_dims % 2 || !(s.rot_base > 0)) { *err = "config: " + mw + "rot"; return false; }
        s.scale = 1.0f / sqrtf(static_cast<float>(s.dim));
        if (jnum(mx, "scale", &d)) s.scale = static_cast<float>(d);
      } else if (ty->str == "delta") {
        s.kind = MIX_DELTA;
        if (given(mx, "conv") && !whole(mx, "conv", 1, &s.taps, mw)) return false;       // otherwise the checkpoint says it
        if (s.dim > 1024) { *err = "config: " + mw + "dim above 1024"; return false; }
      } else { *err = "config: unknown mixer \"" + ty->str + "\""; return false; }
      const JVal* mlp = L.get("mlp");
      if (mlp && mlp->type == JVal::Obj) {
        const JVal* kind = mlp->get("kind");
        if (kind && !(kind->type == JVal::Str && kind->str == "moe")) { *err = "config: " + where + "mlp.kind (moe)"; return false; }
        s.mlp = true;
        const JVal* ro = mlp->get("router");
        if (!whole(ro, "experts", 1, &s.experts, rw) || !whole(ro, "top", 1, &s.top, rw)) return false;
        if (given(ro, "groups")) {
          const JVal* gr = ro->get("groups");
          if (!whole(gr, "count", 1, &s.groups, rw + "groups.") || !whole(gr, "keep", 1, &s.keep, rw + "groups.")) return false;
        }
        if (jnum(ro, "scale", &d)) s.route_scale = static_cast<float>(d);
        if (s.groups > 64 || s.experts % s.groups || s.keep > s.groups || s.top > s.keep * (s.experts / s.groups)) {
          *err = "config: " + rw + "experts, top and groups do not fit each other (at most 64 groups)";
          return false;
        }
        if (given(mlp->get("expert"), "ff") && !whole(mlp->get("expert"), "ff", 1, &s.ff, where + "mlp.expert.")) return false;   // otherwise the checkpoint says it
        if (const JVal* sh = mlp->get("shared")) {
          if (sh->type == JVal::Obj) {
            s.shared = true;
            if (given(sh, "ff") && !whole(sh, "ff", 1, &s.sff, where + "mlp.shared.")) return false;
          }
        }
      }
      layout(s);
      spec.push_back(s);
    }
    run.resize(spec.size());
    return true;
  }

  static int up8(int v) { return (v + 7) / 8 * 8; }
  void layout(LayerSpec& s) {
    int at = 0;
    auto block = [&](int* off, int n) { *off = at; at = up8(at + n); };   // every block starts 16-byte aligned
    const int GD = s.kv_heads * s.dim;
    s.k_out = s.heads * s.vdim;
    if (s.kind == MIX_ATTENTION) {
      block(&s.off_qkv, s.heads * s.dim + GD);
    } else {
      s.conv_c = 2 * GD + s.k_out;
      block(&s.off_qkv, s.conv_c);
      block(&s.off_g, s.k_out);
      block(&s.off_b, s.heads);
      block(&s.off_a, s.heads);
      s.conv_floats = static_cast<size_t>(std::max(s.taps, 1) - 1) * s.conv_c;
      s.rec_floats = static_cast<size_t>(s.heads) * s.dim * s.vdim;
    }
    s.n_in = at;
    s.n_sh = s.shared ? up8(2 * s.sff) : 0;
  }

  int inspect(const CheckpointReader& ck, std::string* err) override {
    std::vector<int64_t> sh;
    for (size_t i = 0; i < spec.size(); ++i) {
      LayerSpec& s = spec[i];
      const std::string p = "l" + std::to_string(i) + ".";
      auto size_of = [&](const std::string& name, int axis, int* out) {
        if (!ck.shape(name, &sh) || sh.size() != 2) { *err = name; return false; }
        *out = static_cast<int>(sh[axis]);
        return true;
      };
      if (s.kind == MIX_DELTA && s.taps == 0 && !size_of(p + "mix.q.conv", 1, &s.taps)) return -4;
      if (s.mlp && s.ff == 0 && !size_of(p + "mlp.e0.gate", 0, &s.ff)) return -4;
      if (s.shared && s.sff == 0 && !size_of(p + "mlp.shared.gate", 0, &s.sff)) return -4;
      layout(s);
    }
    return 0;
  }

  template <typename P>
  int dalloc(P** p, size_t bytes) {
    void* q = nullptr;
    if (cudaMalloc(&q, std::max<size_t>(bytes, 16)) != cudaSuccess) { set_error("Dabodra: device allocation of %zu bytes failed", bytes); return -3; }
    cudaMemsetAsync(q, 0, std::max<size_t>(bytes, 16), env.stream);
    allocs.push_back(q);
    *p = static_cast<P*>(q);
    return 0;
  }

  int init(const ModelEnv& e) override {
    env = e;
    const size_t es = dtype_bytes(dt);
    wts.resize(spec.size());
    int max_in = 8, max_out = 8, max_qn = 0, max_xc = 0, max_rec = 0, max_e = 1, max_top = 1, max_ff = 1, max_nsh = 0, max_sff = 0;
    bool any_moe = false;
    for (size_t i = 0; i < spec.size(); ++i) {
      const LayerSpec& s = spec[i];
      if ((s.kind == MIX_DELTA && s.taps < 1) || (s.mlp && s.ff < 1) || (s.shared && s.sff < 1)) {
        set_error("Dabodra: layer %d: conv, expert.ff or shared.ff is not known", static_cast<int>(i));
        return -1;
      }
      max_in = std::max(max_in, s.n_in); max_out = std::max(max_out, s.k_out);
      if (s.kind == MIX_ATTENTION) max_qn = std::max(max_qn, s.heads * s.dim);
      else { max_xc = std::max(max_xc, s.conv_c); max_rec = std::max(max_rec, s.k_out); }
      if (s.mlp) { any_moe = true; max_e = std::max(max_e, s.experts); max_top = std::max(max_top, s.top); max_ff = std::max(max_ff, s.ff); }
      if (s.shared) { max_nsh = std::max(max_nsh, s.n_sh); max_sff = std::max(max_sff, s.sff); }
    }
    int rc = 0;
    auto mat = [&](void** p, size_t rows, size_t cols) { return dalloc(p, rows * cols * es); };
    auto vec = [&](float** p, size_t n) { return dalloc(p, n * sizeof(float)); };
    rc |= mat(&embed, V, W) | mat(&head, V, W) | vec(&emb_w, W) | vec(&fin_w, W);
    for (size_t i = 0; i < spec.size() && !rc; ++i) {
      const LayerSpec& s = spec[i];
      LayerWeights& w = wts[i];
      LayerRun& r = run[i];
      w.il_e = dt == DT_BF16 && s.mlp && s.ff % 64 == 0;
      w.il_s = dt == DT_BF16 && s.shared && s.sff % 64 == 0;
      rc |= mat(&w.w_in, s.n_in, W) | mat(&w.w_out, W, s.k_out) | vec(&w.norm1, W);
      if (s.kind == MIX_ATTENTION) {
        rc |= vec(&w.q_norm, static_cast<size_t>(s.heads) * s.dim) | vec(&w.k_norm, static_cast<size_t>(s.kv_heads) * s.dim) | vec(&w.sink, s.heads) |
              dalloc(&r.cache, static_cast<size_t>(e.num_blocks) * e.page * 2 * s.kv_heads * s.dim * es);
        if (s.rot_dims) {
          rc |= dalloc(&w.rope, static_cast<size_t>(e.max_model_len) * (s.rot_dims / 2) * sizeof(float2));
          if (!rc && rope_table_yarn(w.rope, e.max_model_len, s.rot_dims, s.rot_base, nullptr, e.stream)) rc = -2;
        }
      } else {
        rc |= vec(&w.conv_w, static_cast<size_t>(s.conv_c) * s.taps) | vec(&w.dt_b, s.heads) | vec(&w.rate, s.heads) | vec(&w.o_norm, s.vdim) |
              vec(&r.conv, e.num_slots * s.conv_floats) | vec(&r.state, e.num_slots * s.rec_floats);
      }
      if (!s.mlp) continue;
      rc |= vec(&w.norm2, W) | mat(&w.router, s.experts, W) | vec(&w.correction, s.experts) | mat(&w.e_gu, static_cast<size_t>(s.experts) * 2 * s.ff, W) |
            mat(&w.e_down, static_cast<size_t>(s.experts) * W, s.ff);
      if (s.shared) rc |= mat(&w.sh_in, s.n_sh, W) | mat(&w.sh_down, W, s.sff);
    }
    if (rc) return rc;
    if (cudaMallocHost(&kernel_error, sizeof(int)) != cudaSuccess) return -3;
    *kernel_error = 0;
    const size_t T = e.Tcap;
    row_cap = static_cast<int>(std::min<size_t>(T, 256));
    rc |= vec(&x, T * W) | mat(&h, T, W) | mat(&inb, T, max_in) | mat(&yb, T, max_out) | mat(&ao, T, W) | mat(&hrow, row_cap, W) |
          vec(&logits, static_cast<size_t>(row_cap) * V);
    if (max_qn) rc |= vec(&qn, T * max_qn);
    if (max_rec) rc |= mat(&xc, T, max_xc) | vec(&o32, T * max_rec);
    if (any_moe) {
      moe_cap = static_cast<int>((T * max_top + 63) / 64 * 64) + max_e * 64;
      rc |= mat(&fo, T, W) | vec(&scores, T * max_e) | vec(&topw, T * max_top) | dalloc(&topi, T * max_top * sizeof(int)) |
            dalloc(&sorted_rows, static_cast<size_t>(moe_cap) * sizeof(int)) | dalloc(&tile_group, static_cast<size_t>(moe_cap / 64) * sizeof(int)) |
            dalloc(&pair_pos, T * max_top * sizeof(int)) | mat(&egu, moe_cap, 2 * static_cast<size_t>(max_ff)) | mat(&eact, moe_cap, max_ff) |
            vec(&edown, static_cast<size_t>(moe_cap) * W) | dalloc(&iota, static_cast<size_t>(64) * sizeof(int));
      if (!rc) {
        int hi[64];
        for (int i = 0; i < 64; ++i) hi[i] = i;
        if (cudaMemcpyAsync(iota, hi, sizeof(hi), cudaMemcpyHostToDevice, e.stream) != cudaSuccess || cudaStreamSynchronize(e.stream) != cudaSuccess) rc = -2;
      }
      if (max_nsh) rc |= mat(&sh, T, max_nsh) | mat(&shact, T, max_sff) | mat(&sdown, T, W);
    }
    if (rc) return rc;
    register_tensors();
    rc = setup_tc();
    if (rc) return rc;
    return cudaStreamSynchronize(e.stream) == cudaSuccess ? 0 : -2;
  }

  // The projections of a bf16 model run on the tcgen05 pair GEMM (gemm2_tcgen05.cu) where their shapes allow it (rows and
  // columns in multiples of 8): input and output projection and the shared expert; the routed experts on its grouped form
  // (gemm_grouped.cu).  B200_DB_TC=0 keeps everything on linear.cu (A/B knob); fp32 models always do.
  int setup_tc() {
    const char* ev = getenv("B200_DB_TC");
    use_tc = dt == DT_BF16 && !(ev && atoi(ev) == 0) && W % 8 == 0 && gemm_variant() == 2;
    if (!use_tc) return 0;
    int maxN = W;
    for (auto& s : spec) maxN = std::max(std::max(maxN, s.n_in), std::max(s.n_sh, 2 * s.ff));
    const size_t ws_bytes = std::max(gemm_workspace_bytes(env.sms), gemm_deferred_ws_bytes(env.sms));
    if (dalloc(&gemm_ws, ws_bytes)) return -3;
    const size_t n_counters = 2ull * (maxN / 128 + 2) * (env.Tcap / 32 + 2);
    if (dalloc(&gemm_counters, n_counters * sizeof(int))) return -3;
    if (const char* e = getenv("B200_DB_FEW_ROWS")) few_rows = atoi(e);            // A/B knobs
    if (const char* e = getenv("B200_DB_WHOLE")) whole = atoi(e) != 0;
    bool grouped = true;
    if (const char* e = getenv("B200_DB_GROUPED")) grouped = atoi(e) != 0;
    const int bns[kGemmNumBlockN] = {32, 64, 128, 256, 512};
    auto maps = [&](CUtensorMap* m, const void* X, int K) {
      for (int i = 0; i < kGemmNumBlockN; ++i)
        if (gemm_make_x_map(&m[i], X, env.Tcap, K, K, bns[i])) return false;
      return true;
    };
    auto plan = [&](GemmPlan* p, const void* Wm, int N, int K) {
      if (N % 8 || K % 8 || gemm_plan_init(p, Wm, N, K, K, gemm_ws, gemm_counters, env.sms)) return false;
      p->ws_bytes = ws_bytes;
      return true;
    };
    auto plan_maps = [&](GemmPlan* p, CUtensorMap* m, const void* X, const void* Wm, int N, int K) {
      if (!plan(p, Wm, N, K)) return false;
      if (maps(m, X, K)) return true;
      gemm_plan_destroy(p);
      return false;
    };
    if (!maps(xm_h, h, W)) { use_tc = false; return 0; }
    int max_e = 1;
    bool any_mlp = false;
    for (auto& s : spec)
      if (s.mlp) { any_mlp = true; max_e = std::max(max_e, s.experts); }
    if (any_mlp && (dalloc(&hsorted, static_cast<size_t>(moe_cap) * W * 2) || dalloc(&edown16, static_cast<size_t>(moe_cap) * W * 2) ||
                    dalloc(&expert_rows, static_cast<size_t>(max_e) * 2 * sizeof(int)))) return -3;
    for (size_t i = 0; i < spec.size(); ++i) {
      const LayerSpec& s = spec[i];
      LayerWeights& w = wts[i];
      w.tc_in = plan(&w.p_in, w.w_in, s.n_in, W);
      w.tc_out = plan_maps(&w.p_out, w.xm_out, yb, w.w_out, W, s.k_out);
      if (s.shared) {
        w.tc_shin = plan(&w.p_shin, w.sh_in, s.n_sh, W);
        w.tc_shdown = plan_maps(&w.p_shdown, w.xm_shact, shact, w.sh_down, W, s.sff);
      }
      if (s.mlp && grouped)
        w.tc_experts = !gemm_grouped_plan(&w.g_egu, w.e_gu, s.experts, 2 * s.ff, W) && !gemm_grouped_plan(&w.g_edown, w.e_down, s.experts, W, s.ff) &&
                       !gemm_grouped_x_map(&w.xg_h, hsorted, moe_cap, W) && !gemm_grouped_x_map(&w.xg_act, eact, moe_cap, s.ff);
    }
    return 0;
  }

  void reg(const std::string& name, void* p, size_t bytes) { tensors[name] = {p, bytes}; }
  void register_tensors() {
    const size_t es = dtype_bytes(dt);
    reg("embed", embed, static_cast<size_t>(V) * W * es);
    reg("head", head, static_cast<size_t>(V) * W * es);
    for (size_t i = 0; i < spec.size(); ++i) {
      const std::string p = "l" + std::to_string(i) + ".";
      reg(p + "w_in", wts[i].w_in, static_cast<size_t>(spec[i].n_in) * W * es);
      reg(p + "w_out", wts[i].w_out, static_cast<size_t>(W) * spec[i].k_out * es);
    }
  }

  // ------------------------------------------------------------ weights
  // host fp32 [rows, cols] -> device rows [row0, row0 + rows) of a matrix with `cols` columns
  int put(void* dst, size_t row0, const std::vector<float>& src, size_t rows, size_t cols) {
    const size_t es = dtype_bytes(dt);
    std::vector<uint8_t> tmp(rows * cols * es);
    if (dt == DT_F32) memcpy(tmp.data(), src.data(), tmp.size());
    else {
      bf16* o = reinterpret_cast<bf16*>(tmp.data());
      for (size_t i = 0; i < rows * cols; ++i) o[i] = __float2bfloat16_rn(src[i]);
    }
    return cudaMemcpy(static_cast<uint8_t*>(dst) + row0 * cols * es, tmp.data(), tmp.size(), cudaMemcpyHostToDevice) == cudaSuccess ? 0 : -2;
  }
  // gate and up rows [F, cols] each, one below the other or in alternating blocks of 64
  int put_pair(void* dst, size_t row0, const std::vector<float>& gate, const std::vector<float>& up, size_t F, size_t cols, bool in_turns) {
    std::vector<float> both;
    both.reserve(2 * F * cols);
    const size_t block = (in_turns ? 64 : F) * cols;
    for (size_t at = 0; at < F * cols; at += block) {
      both.insert(both.end(), gate.begin() + at, gate.begin() + at + block);
      both.insert(both.end(), up.begin() + at, up.begin() + at + block);
    }
    return put(dst, row0, both, 2 * F, cols);
  }
  int putf(float* dst, const std::vector<float>& src) {
    return cudaMemcpy(dst, src.data(), src.size() * sizeof(float), cudaMemcpyHostToDevice) == cudaSuccess ? 0 : -2;
  }

  int load(const CheckpointReader& ck, std::string* err) override {
    std::vector<float> v;
    std::vector<int64_t> sh;
    auto get = [&](const std::string& name, int64_t rows, int64_t cols) {
      if (!ck.read_f32(name, &v, &sh, err)) return false;
      int64_t n = 1;
      for (auto d : sh) n *= d;
      const int64_t r = sh.size() == 2 ? sh[0] : 1, c = sh.size() == 2 ? sh[1] : n;
      if (r != rows || c != cols) {
        *err = name + ": shape [" + std::to_string(r) + "," + std::to_string(c) + "] does not fit the config";
        return false;
      }
      return true;
    };
    int rc = 0;
#define MAT(name, dst, row0, rows, cols) do { if (!get(name, rows, cols)) return -4; rc |= put(dst, row0, v, rows, cols); } while (0)
#define PAIR(prefix, dst, row0, F, cols, turns) do { if (!get((prefix) + "gate", F, cols)) return -4; const std::vector<float> g_ = v; \
    if (!get((prefix) + "up", F, cols)) return -4; rc |= put_pair(dst, row0, g_, v, F, cols, turns); } while (0)
#define VEC(name, dst, n) do { if (!get(name, 1, n)) return -4; rc |= putf(dst, v); } while (0)
#define NORM(name, dst, n) do { if (!get(name, 1, n)) return -4; for (auto& e_ : v) e_ += 1.0f; rc |= putf(dst, v); } while (0)   // stored as the offset from one
    MAT("embed", embed, 0, V, W);
    MAT("head", head, 0, V, W);
    NORM("embed.norm", emb_w, W);
    NORM("final.norm", fin_w, W);
    for (size_t i = 0; i < spec.size(); ++i) {
      const LayerSpec& s = spec[i];
      LayerWeights& w = wts[i];
      const std::string p = "l" + std::to_string(i) + ".", mx = p + "mix.", f = p + "mlp.";
      const int HD = s.heads * s.dim, GD = s.kv_heads * s.dim, HV = s.k_out;
      NORM(p + "norm1", w.norm1, W);
      if (s.kind == MIX_ATTENTION) {
        MAT(mx + "q", w.w_in, s.off_qkv, HD, W);
        MAT(mx + "k", w.w_in, s.off_qkv + HD, GD, W);
        VEC(mx + "q.norm", w.q_norm, HD);
        VEC(mx + "k.norm", w.k_norm, GD);
        VEC(mx + "sink", w.sink, s.heads);
      } else {
        MAT(mx + "q", w.w_in, s.off_qkv, GD, W);
        MAT(mx + "k", w.w_in, s.off_qkv + GD, GD, W);
        MAT(mx + "v", w.w_in, s.off_qkv + 2 * GD, HV, W);
        MAT(mx + "g", w.w_in, s.off_g, HV, W);
        MAT(mx + "b", w.w_in, s.off_b, s.heads, W);
        MAT(mx + "a", w.w_in, s.off_a, s.heads, W);
        std::vector<float> taps;
        const struct { const char* name; int rows; } conv[3] = {{"q.conv", GD}, {"k.conv", GD}, {"v.conv", HV}};
        for (auto& cv : conv) {
          if (!get(mx + cv.name, cv.rows, s.taps)) return -4;
          taps.insert(taps.end(), v.begin(), v.end());
        }
        rc |= putf(w.conv_w, taps);
        VEC(mx + "dt_bias", w.dt_b, s.heads);
        if (!get(mx + "A_log", 1, s.heads)) return -4;
        for (auto& a : v) a = static_cast<float>(-exp(static_cast<double>(a)));     // the decay's rate, once
        rc |= putf(w.rate, v);
        VEC(mx + "norm", w.o_norm, s.vdim);
      }
      MAT(mx + "o", w.w_out, 0, W, HV);
      if (!s.mlp) continue;
      NORM(p + "norm2", w.norm2, W);
      MAT(f + "router", w.router, 0, s.experts, W);
      VEC(f + "correction", w.correction, s.experts);
      for (int e = 0; e < s.experts; ++e) {
        const std::string ep = f + "e" + std::to_string(e) + ".";
        PAIR(ep, w.e_gu, static_cast<size_t>(e) * 2 * s.ff, s.ff, W, w.il_e);
        MAT(ep + "down", w.e_down, static_cast<size_t>(e) * W, W, s.ff);
      }
      if (s.shared) {
        PAIR(f + "shared.", w.sh_in, 0, s.sff, W, w.il_s);
        MAT(f + "shared.down", w.sh_down, 0, W, s.sff);
      }
    }
#undef MAT
#undef PAIR
#undef VEC
#undef NORM
    if (rc) { *err = "copying weights to the device failed"; return -2; }
    return 0;
  }

  // Seeded random weights of a plausible scale (benchmarks: there is no checkpoint of a real size).
  int randomize(uint64_t seed) override {
    cudaStream_t st = env.stream;
    int rc = 0;
    uint64_t k = seed * 1000003ull + 71;
    auto M = [&](void* p, size_t n, float sc) { if (p) rc |= fill_uniform(p, dt, n, ++k, sc, 0.f, st); };
    auto F = [&](float* p, size_t n, float sc, float off) { if (p) rc |= fill_uniform(p, DT_F32, n, ++k, sc, off, st); };
    auto by = [](int n) { return 1.7f / sqrtf(static_cast<float>(n)); };
    M(embed, static_cast<size_t>(V) * W, 1.f);
    M(head, static_cast<size_t>(V) * W, by(W));
    F(emb_w, W, 0.1f, 1.f); F(fin_w, W, 0.1f, 1.f);
    for (size_t i = 0; i < spec.size(); ++i) {
      const LayerSpec& s = spec[i];
      LayerWeights& w = wts[i];
      M(w.w_in, static_cast<size_t>(s.n_in) * W, by(W));
      M(w.w_out, static_cast<size_t>(W) * s.k_out, by(s.k_out));
      F(w.norm1, W, 0.1f, 0.5f); F(w.norm2, W, 0.1f, 0.5f);
      if (s.kind == MIX_ATTENTION) {
        F(w.q_norm, static_cast<size_t>(s.heads) * s.dim, 0.1f, 1.f); F(w.k_norm, static_cast<size_t>(s.kv_heads) * s.dim, 0.1f, 1.f); F(w.sink, s.heads, 1.f, 0.f);
      } else {
        F(w.conv_w, static_cast<size_t>(s.conv_c) * s.taps, 0.5f, 0.3f); F(w.dt_b, s.heads, 1.f, -3.f); F(w.rate, s.heads, 0.4f, -0.5f); F(w.o_norm, s.vdim, 0.1f, 1.f);
      }
      if (!s.mlp) continue;
      M(w.router, static_cast<size_t>(s.experts) * W, by(W)); F(w.correction, s.experts, 0.05f, 0.f);
      M(w.e_gu, static_cast<size_t>(s.experts) * 2 * s.ff * W, by(W));
      M(w.e_down, static_cast<size_t>(s.experts) * W * s.ff, by(s.ff));
      if (s.shared) { M(w.sh_in, static_cast<size_t>(s.n_sh) * W, by(W)); M(w.sh_down, static_cast<size_t>(W) * s.sff, by(s.sff)); }
    }
    if (rc) return -2;
    return cudaStreamSynchronize(st) == cudaSuccess ? 0 : -2;
  }

  // ------------------------------------------------------------ forward
  // Y = X W^T.  Steps of up to 16 tokens stream the weights through linear.cu's fragment kernel, steps of up to 256 tokens take
  // the stream-K pair GEMM (every weight byte once, all pairs busy), larger ones whole tiles.
  // The grouped kernel on one matrix: whole 256 x 256 tiles, the accumulator drained under the next tile.
  bool takes_whole(bool tc, int T) const { return tc && T > 256 && whole; }
  int run_whole(const GemmPlan& plan, const CUtensorMap* xm, bool glu, void* Y, int ldy, int T) {
    GroupedPlan g;
    g.tm_w = plan.tm_w; g.experts = 1; g.N = plan.N; g.K = plan.K;      // the same boxes: 128 rows x 64 columns on both sides
    return gemm_grouped_run(g, xm[gemm_block_n_index(256)], nullptr, Y, ldy, glu, env.sms, kernel_error, env.stream, T);
  }
  int project(const GemmPlan& plan, bool tc, const CUtensorMap* xm, const void* X, const void* Wm, void* Y, int T, int N, int K) {
    if (takes_whole(tc, T)) return run_whole(plan, xm, false, Y, N, T);
    if (tc && T > few_rows) {
      const int bn = gemm_block_n_for(T);
      return gemm_run(plan, xm[gemm_block_n_index(bn)], bn, Y, N, T, env.stream);
    }
    return linear(linear_args(X, dt, Wm, dt, Y, dt, T, N, K), env.stream);
  }
  // per-kernel device time (b200_engine_kernel_times): with profiling on, every launch is bracketed by events and waited for
  cudaEvent_t pe0 = nullptr, pe1 = nullptr;
  void prof_start() {
    if (!profile_kernels) return;
    if (!pe0) { cudaEventCreate(&pe0); cudaEventCreate(&pe1); }
    cudaEventRecord(pe0, env.stream);
  }
  void prof_stop(const char* name) {
    if (!profile_kernels) return;
    cudaEventRecord(pe1, env.stream);
    cudaEventSynchronize(pe1);
    float ms = 0.f;
    cudaEventElapsedTime(&ms, pe0, pe1);
    auto& t = kernel_times[name];
    t.first += ms * 1000.0;
    t.second += 1;
  }
#define KRN(name, call) do { prof_start(); const int r_ = (call); if (r_ && !rc) { failed_kernel = name; failed_rc = r_; } rc |= r_; prof_stop(name); ++nl; } while (0)
  const char* failed_kernel = "";
  int failed_rc = 0;

  void* col(void* base, size_t off) const { return static_cast<uint8_t*>(base) + off * dtype_bytes(dt); }

  // the output of the last sublayer, still to be normed and added by the next boundary
  struct Pending {
    const void* y = nullptr;
    const float* post_w = nullptr;
  };
  SandwichArgs boundary(const Pending& p, const float* pre_w, void* out, const int* row_index, int rows) {
    SandwichArgs a;
    a.x = x; a.y = p.y; a.ty = dt; a.y_bias = nullptr;
    a.post_w = p.post_w; a.pre_w = pre_w; a.eps = eps;
    a.h = out; a.th = dt; a.row_index = row_index; a.rows = rows; a.W = W;
    return a;
  }

  int mix_attention(const LayerSpec& s, const LayerWeights& w, const LayerRun& r, const StepBatch& b, int64_t& nl) {
    cudaStream_t st = env.stream;
    int rc = 0;
    ConvQkPrepArgs qp = {};
    qp.qk = col(inb, s.off_qkv); qp.ld = s.n_in; qp.t = dt;
    qp.q_norm_w = w.q_norm; qp.k_norm_w = w.k_norm; qp.eps = eps;
    qp.rope = w.rope; qp.rot_dims = s.rot_dims; qp.interleaved = true;
    qp.positions = b.pos; qp.slots = b.slots; qp.seq_of_tok = b.seq_of_tok; qp.seqs = b.seqs;
    qp.qn = qn; qp.cache = r.cache;
    qp.T = b.T; qp.heads = s.heads; qp.kv_heads = s.kv_heads; qp.dim = s.dim;
    KRN("qk_prep", conv_qk_prep(qp, st));
    WindowAttnArgs wa = {};
    wa.qn = qn; wa.cache = r.cache; wa.t = dt; wa.positions = b.pos; wa.seq_of_tok = b.seq_of_tok; wa.block_tables = b.btab;
    wa.max_blocks = b.max_blocks; wa.page = env.page;
    wa.out_scale = 1.f; wa.y = yb; wa.ldy = s.k_out;
    wa.T = b.T; wa.heads = s.heads; wa.kv_heads = s.kv_heads; wa.dim = s.dim; wa.vdim = s.vdim;
    wa.window = s.window; wa.scale = s.scale; wa.sink = w.sink;
    wa.seqs = b.seqs; wa.nseq = b.nseq; wa.max_ctx = b.max_ctx;
    KRN("window_attention", window_attention(wa, st));
    return rc;
  }

  int mix_delta(const LayerSpec& s, const LayerWeights& w, const LayerRun& r, const StepBatch& b, int64_t& nl) {
    cudaStream_t st = env.stream;
    const int GD = s.kv_heads * s.dim;
    int rc = 0;
    ShortConvArgs cc = {};
    cc.u = col(inb, s.off_qkv); cc.ldu = s.n_in; cc.t = dt; cc.w = w.conv_w; cc.act = CONV_SILU;
    cc.y = xc; cc.ldy = s.conv_c; cc.ty = dt; cc.state = r.conv;
    cc.seq_of_tok = b.seq_of_tok; cc.seqs = b.seqs; cc.nseq = b.nseq; cc.T = b.T; cc.C = s.conv_c; cc.taps = s.taps;
    KRN("short_conv", short_conv(cc, st));
    if (s.taps > 1) KRN("conv_carry", short_conv_carry(cc, st));
    DeltaArgs d = {};
    d.qkv = xc; d.t = dt; d.ld = s.conv_c; d.q_off = 0; d.k_off = GD; d.v_off = 2 * GD;
    d.beta_pre = col(inb, s.off_b); d.dt_pre = col(inb, s.off_a); d.ld_gate = s.n_in;
    d.dt_bias = w.dt_b; d.rate = w.rate;
    d.q_scale = 1.0f / sqrtf(static_cast<float>(s.dim)); d.unit_eps = kUnitEps;
    d.states = r.state; d.seqs = b.seqs; d.nseq = b.nseq; d.T = b.T;
    d.heads = s.heads; d.kv_heads = s.kv_heads; d.dim = s.dim; d.vdim = s.vdim; d.o = o32;
    KRN("delta_scan", delta_scan(d, st));
    OutGateArgs og = {};
    og.o = o32; og.g = col(inb, s.off_g); og.ldg = s.n_in; og.w = w.o_norm; og.eps = eps;
    og.y = yb; og.ldy = s.k_out; og.t = dt; og.T = b.T; og.heads = s.heads; og.vdim = s.vdim;
    og.joint = false; og.gate_act = GATE_SILU; og.out_scale = 1.f;
    KRN("delta_out_gate", recurrent_out_gate(og, st));
    return rc;
  }

  int moe(const LayerSpec& s, const LayerWeights& w, int T, int64_t& nl) {
    cudaStream_t st = env.stream;
    int rc = 0;
    KRN("moe_router", linear(linear_args(h, dt, w.router, dt, scores, DT_F32, T, s.experts, W), st));
    MoeRouteForm form;
    form.group_best = 2; form.normalize = true; form.sum_eps = kWeightSumEps; form.scale = s.route_scale;
    KRN("moe_route", moe_route(scores, topi, topw, T, s.experts, s.groups, s.keep, s.top, st, MOE_SIGMOID, s.experts, w.correction, form));
    const void* shared_out = nullptr;
    if (s.shared) {
      if (w.il_s && takes_whole(w.tc_shin, T)) {
        KRN("shared_in", run_whole(w.p_shin, xm_h, true, shact, s.sff, T));     // the gated unit in the epilogue
      } else {
        KRN("shared_in", project(w.p_shin, w.tc_shin, xm_h, h, w.sh_in, sh, T, s.n_sh, W));
        KRN("glu", glu_clamped(sh, s.n_sh, shact, s.sff, dt, T, s.sff, INFINITY, 1.f, st, 0.f, w.il_s));
      }
      KRN("shared_down", project(w.p_shdown, w.tc_shdown, w.xm_shact, shact, w.sh_down, sdown, T, W, s.sff));
      shared_out = sdown;
    }
    const long long gu_stride = 2ll * s.ff * W, down_stride = static_cast<long long>(W) * s.ff;
    if (T * s.top <= 64) {
      // decode-sized steps: one weight-streaming pass per chosen (token, expert) pair, rows in pair order
      LinearArgs up = linear_args(h, dt, w.e_gu, dt, egu, dt, T * s.top, 2 * s.ff, W);
      up.wbs = gu_stride;
      const PickedRows pu = {T * s.top, nullptr, s.top, iota, topi};
      KRN("moe_up", linear_picked_rows(up, pu, st));
      KRN("glu", glu_clamped(egu, 2 * s.ff, eact, s.ff, dt, T * s.top, s.ff, INFINITY, 1.f, st, 0.f, w.il_e));
      LinearArgs dn = linear_args(eact, dt, w.e_down, dt, edown, DT_F32, T * s.top, W, s.ff);
      dn.wbs = down_stride;
      const PickedRows pd = {T * s.top, iota, 1, iota, topi};
      KRN("moe_down", linear_picked_rows(dn, pd, st));
      // pair k of token t is row t * top + k: the combine walks them through an identity table
      KRN("moe_combine", moe_combine_add(edown, DT_F32, iota, topw, shared_out, nullptr, 0, fo, dt, T, s.top, W, st));
      return rc;
    }
    const int cap = (T * s.top + 63) / 64 * 64 + s.experts * 64;
    KRN("moe_align", moe_align(topi, T, s.top, s.experts, sorted_rows, tile_group, pair_pos, cap, st, w.tc_experts ? expert_rows : nullptr));
    if (w.tc_experts) {
      // the inputs in expert-sorted order, then one grouped GEMM per matrix; the row counts stay on the device
      KRN("moe_gather", moe_gather_bf16(h, sorted_rows, hsorted, cap, W, st));
      if (w.il_e) {
        KRN("moe_up", gemm_grouped_run(w.g_egu, w.xg_h, expert_rows, eact, s.ff, true, env.sms, kernel_error, st));
      } else {
        KRN("moe_up", gemm_grouped_run(w.g_egu, w.xg_h, expert_rows, egu, 2 * s.ff, false, env.sms, kernel_error, st));
        KRN("glu", glu_clamped(egu, 2 * s.ff, eact, s.ff, dt, cap, s.ff, INFINITY, 1.f, st, 0.f));
      }
      KRN("moe_down", gemm_grouped_run(w.g_edown, w.xg_act, expert_rows, edown16, W, false, env.sms, kernel_error, st));
      KRN("moe_combine", moe_combine_add(edown16, DT_BF16, pair_pos, topw, shared_out, nullptr, 0, fo, dt, T, s.top, W, st));
      return rc;
    }
    LinearArgs up = linear_args(h, dt, w.e_gu, dt, egu, dt, cap, 2 * s.ff, W);
    up.x_rows = sorted_rows; up.tile_group = tile_group; up.wbs = gu_stride;
    KRN("moe_up", linear(up, st));
    KRN("glu", glu_clamped(egu, 2 * s.ff, eact, s.ff, dt, cap, s.ff, INFINITY, 1.f, st, 0.f, w.il_e));
    LinearArgs dn = linear_args(eact, dt, w.e_down, dt, edown, DT_F32, cap, W, s.ff);
    dn.tile_group = tile_group; dn.wbs = down_stride;
    KRN("moe_down", linear(dn, st));
    KRN("moe_combine", moe_combine_add(edown, DT_F32, pair_pos, topw, shared_out, nullptr, 0, fo, dt, T, s.top, W, st));
    return rc;
  }

  int forward(const StepBatch& b, int* sampled, float* host_logits, int64_t* launches) override {
    cudaStream_t st = env.stream;
    const int T = b.T;
    int rc = 0;
    int64_t nl = 0;
    if (kernel_error && *static_cast<volatile int*>(kernel_error)) { set_error("Dabodra forward: a wait inside the grouped GEMM ran out"); return -2; }
    KRN("embed", embed_normed(embed, dt, b.ids, emb_w, eps, x, h, dt, T, W, V, st));
    Pending pend;
    for (size_t li = 0; li < spec.size() && !rc; ++li) {
      const LayerSpec& s = spec[li];
      const LayerWeights& w = wts[li];
      const LayerRun& r = run[li];
      if (li > 0) KRN("residual_norm", sandwich_step(boundary(pend, nullptr, h, nullptr, T), st));   // layer 0 reads what the embedding left
      KRN("proj_in", project(w.p_in, w.tc_in, xm_h, h, w.w_in, inb, T, s.n_in, W));
      rc |= s.kind == MIX_ATTENTION ? mix_attention(s, w, r, b, nl) : mix_delta(s, w, r, b, nl);
      KRN("proj_out", project(w.p_out, w.tc_out, w.xm_out, yb, w.w_out, ao, T, W, s.k_out));
      pend.y = ao; pend.post_w = w.norm1;
      if (s.mlp) {
        KRN("residual_norm", sandwich_step(boundary(pend, nullptr, h, nullptr, T), st));
        rc |= moe(s, w, T, nl);
        pend.y = fo; pend.post_w = w.norm2;
      }
      if (residual_sink && !rc) {
        // debug: apply the write-back now and read the residual
        KRN("residual_norm", sandwich_step(boundary(pend, nullptr, nullptr, nullptr, T), st));
        pend = Pending();
        const size_t at = residual_sink->size();
        residual_sink->resize(at + static_cast<size_t>(T) * W);
        if (rc || cudaMemcpyAsync(residual_sink->data() + at, x, static_cast<size_t>(T) * W * sizeof(float), cudaMemcpyDeviceToHost, st) != cudaSuccess ||
            cudaStreamSynchronize(st) != cudaSuccess) rc = -2;
      }
    }
    if (pend.y) KRN("residual_norm", sandwich_step(boundary(pend, nullptr, nullptr, nullptr, T), st));
    // head: the last norm over the wanted rows, logits in fp32, greedy choice
    for (int r0 = 0; r0 < b.S && !rc; r0 += row_cap) {
      const int n = std::min(row_cap, b.S - r0);
      KRN("residual_norm", sandwich_step(boundary(Pending(), fin_w, hrow, b.rows + r0, n), st));
      KRN("head", linear(linear_args(hrow, dt, head, dt, logits, DT_F32, n, V, W), st));
      KRN("argmax", argmax_f32(logits, sampled + r0, n, V, st));
      if (host_logits && cudaMemcpyAsync(host_logits + static_cast<size_t>(r0) * V, logits, static_cast<size_t>(n) * V * sizeof(float),
                                         cudaMemcpyDeviceToHost, st) != cudaSuccess) rc = -2;
    }
    if (launches) *launches += nl;
    if (rc) { set_error("Dabodra forward: %s failed with %d (%s)", failed_kernel, failed_rc, cudaGetErrorString(cudaGetLastError())); return -2; }
    return 0;
  }
};

}  // namespace

#undef KRN

std::unique_ptr<Model> make_dabodra(const JVal& config, DType dtype, std::string* err) {
  std::unique_ptr<Dabodra> m(new Dabodra(dtype));
  if (!m->parse(config, err)) return nullptr;
  return std::unique_ptr<Model>(m.release());
}

}  // namespace b200
