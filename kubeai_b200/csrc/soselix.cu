// Soselix: a decoder-only pre-norm design on one fp32 residual with a residual multiplier, whose layers mix tokens by
// latent attention, by the HGRN2 recurrence or by Mamba-2, and whose feed-forward is one biased hidden layer under xIELU.
//
//   x[t]     = embed[token] * embedding.scale
//   sublayer : h = g * x / rms(x)  (ONE learned number g per norm);  x <- x + m f(h),  m = residual_mult     (sandwich_step)
//   latent_attention: cq = rmsnorm(W_dq h), q = W_uq cq (per head: dim unrotated, rot_dim rotated dimensions);
//              [c | kr] = W_dkv h, c RMS-normed, kr rotated: both cached, shared by the heads; per head
//              score_j = (q . W_uk c_j + rot(q') . kr_j) * scale, causal softmax with exp(sink_h) in its denominator,
//              W_uv on the weighted sum of the c_j, times sigmoid(W_g h)_h, W_o; rotation pairs (i, i + rot.dims / 2).
//              With `kv_from`: j the layer has no W_dkv and reads the cache rows of layer j   (latent_attention.cu, absorbed form)
//   hgrn2    : f = l + (1 - l) sigmoid(W_f h + b), S <- diag(f) S + (1 - f) v^T, o = S^T silu(W_q h); every head's o RMS-normed
//              with one shared weight, W_o                                                       (gla.cu, fgate_lower form)
//   mamba2   : [z | x | B | C | dt] = W_in h; x, B, C pass a short causal convolution and SiLU; d = softplus(dt + b);
//              S <- exp(-exp(A_log) d) S + d B x^T, y = S^T C + D x (B, C shared by the heads of a group); y * silu(z), RMS norm
//              in norm_groups parts, W_o                                   (ssm.cu, gla.cu: dt_pre form, gated_group_norm)
//   ff       : W_down xIELU(W_up h + b_up) + b_down                                                   (bias_act)
//   logits   = head (g_f * x / rms(x))
//
// Per layer the kernel sequence is: the residual boundary (previous write-back + norm), ONE input projection for everything
// that reads the mixer's input, the mixer's own kernels, its output projection, and for the feed-forward a boundary, the
// up-projection, bias + activation in place, and the down-projection, whose bias rides in the next boundary.  Every size
// and constant comes from config.json; matrices and activations are bf16 or fp32; the residual, norms, softmax, gates of
// the recurrences, decays and recurrent states are fp32 either way.  A sequence's state slot holds the carried convolution
// inputs and the recurrent state of every recurrent layer; the page pool holds the latent rows of every attention layer
// that makes its own.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <string.h>

#include <algorithm>

#include "epi_pass.cuh"
#include "errors.h"
#include "gemm.h"
#include "model.h"

namespace b200 {
namespace {

typedef __nv_bfloat16 bf16;

enum MixerKind { MIX_LATENT = 0, MIX_HGRN2 = 1, MIX_MAMBA2 = 2 };

struct LayerSpec {
  int kind = MIX_LATENT;
  int heads = 0, dim = 0, vdim = 0;
  // latent attention
  int rot_dim = 0, kv_rank = 0, q_rank = 0, rot_dims = 0, kv_from = -1;
  double rot_base = 10000.0;
  float scale = 1.f;
  // mamba2 (dim is the state size)
  int groups = 1, norm_groups = 1, taps = 1;
  bool mlp = false;
  int ff = 0;
  // column layout of the input projection's output row
  int n_in = 0, off_dq = 0, off_dkv = 0, off_g = 0, off_q = 0, off_f = 0, off_v = 0, off_z = 0, off_xbc = 0, off_dt = 0;
  int k_out = 0, conv_c = 0;
  size_t conv_floats = 0, rec_floats = 0;   // the layer's part of a state slot: carried convolution inputs, recurrent state
  bool own_cache() const { return kind == MIX_LATENT && kv_from < 0; }
};

struct LayerWeights {
  void* w_in = nullptr;     // [n_in, width]
  void* w_out = nullptr;    // [width, k_out]
  void *w_uq = nullptr, *uk_t = nullptr, *w_uv = nullptr;   // [heads (dim + rot_dim), q_rank], [heads][kv_rank][dim], [heads][vdim][kv_rank]
  void *w_up = nullptr, *w_down = nullptr;                  // [ff, width], [width, ff]
  float *norm1 = nullptr, *norm2 = nullptr;                 // the norm's one number, spread over the width
  float *cq_norm = nullptr, *c_norm = nullptr, *sink = nullptr;
  float2* rope = nullptr;
  float *f_b = nullptr, *lower = nullptr, *o_norm = nullptr;   // o_norm: [vdim] (hgrn2) or [heads * vdim] (mamba2)
  float *conv_w = nullptr, *conv_b = nullptr, *dt_b = nullptr, *dt_rate = nullptr, *skip = nullptr;
  float *up_b = nullptr, *down_b = nullptr;
  float act_pos = 0.f, act_neg = 0.f;
  GemmPlan p_in, p_out, p_uq, p_up, p_down;
  CUtensorMap xm_out[kGemmNumBlockN], xm_cq[kGemmNumBlockN], xm_hid[kGemmNumBlockN];
  bool tc_in = false, tc_out = false, tc_uq = false, tc_up = false, tc_down = false;
};

struct LayerRun {
  void* cache = nullptr;    // latent attention with its own rows: [num_blocks * page][kv_rank + rot_dim]
  float* conv = nullptr;    // [slots][taps - 1][channels]: the carried inputs of the layer's convolution
  float* state = nullptr;   // [slots][heads][dim][vdim]
};

bool jnum(const JVal* o, const char* k, double* out) {
  const JVal* v = o ? o->get(k) : nullptr;
  if (!v || v->type != JVal::Num) return false;
  *out = v->num;
  return true;
}

class Soselix : public Model {
 public:
  DType dt;
  int V = 0, W = 0;
  float eps = 1e-5f, mult = 1.f, embed_scale = 1.f;
  std::vector<LayerSpec> spec;
  std::vector<LayerWeights> wts;
  std::vector<LayerRun> run;
  ModelEnv env;
  void *embed = nullptr, *head = nullptr;
  float* fin_w = nullptr;
  // activations
  float *x = nullptr, *o32 = nullptr, *qlat = nullptr, *olat = nullptr, *logits = nullptr, *split_ws = nullptr;
  long long split_ws_floats = 0;
  void *h = nullptr, *inb = nullptr, *cq = nullptr, *qb = nullptr, *xc = nullptr, *yb = nullptr, *ao = nullptr, *hid = nullptr, *fo = nullptr, *hrow = nullptr;
  int row_cap = 0;
  std::vector<void*> allocs;
  float* gemm_ws = nullptr;
  int* gemm_counters = nullptr;
  int* gemm_flags = nullptr;     // of the fused form: two per CTA pair, stamped with the launch's number
  int gemm_epoch = 0;
  bool fuse = true;
  int few_rows = 16;
  CUtensorMap xm_h[kGemmNumBlockN];
  bool use_tc = false;

  explicit Soselix(DType d) : dt(d) {}
  ~Soselix() override {
    for (auto& w : wts) {
      if (w.tc_in) gemm_plan_destroy(&w.p_in);
      if (w.tc_out) gemm_plan_destroy(&w.p_out);
      if (w.tc_uq) gemm_plan_destroy(&w.p_uq);
      if (w.tc_up) gemm_plan_destroy(&w.p_up);
      if (w.tc_down) gemm_plan_destroy(&w.p_down);
    }
    if (pe0) { cudaEventDestroy(pe0); cudaEventDestroy(pe1); }
    for (void* p : allocs) cudaFree(p);
  }
  const char* arch() const override { return "Soselix"; }
  int vocab() const override { return V; }

  size_t cache_bytes_per_block(int page) const override {
    size_t b = 0;
    for (auto& s : spec)
      if (s.own_cache()) b += static_cast<size_t>(page) * (s.kv_rank + s.rot_dim) * dtype_bytes(dt);
    return b;
  }
  size_t state_bytes_per_slot() const override {
    size_t b = 0;
    for (auto& s : spec) b += (s.conv_floats + s.rec_floats) * sizeof(float);
    return b;
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
    auto given = [](const JVal* o, const char* k) { const JVal* v = o->get(k); return v && !v->is_null(); };
    if (!whole(&c, "vocab", 1, &V, "") || !whole(&c, "width", 1, &W, "")) return false;
    if (W > 12288) { *err = "config: width above 12288"; return false; }
    if (jnum(c.get("norm"), "eps", &d)) eps = static_cast<float>(d);
    if (jnum(&c, "residual_mult", &d)) mult = static_cast<float>(d);
    if (jnum(c.get("embedding"), "scale", &d)) embed_scale = static_cast<float>(d);
    const JVal* ls = c.get("layers");
    if (!ls || ls->type != JVal::Arr || ls->arr.empty()) { *err = "config: layers"; return false; }
    for (size_t i = 0; i < ls->arr.size(); ++i) {
      const JVal& L = ls->arr[i];
      const std::string where = "layer " + std::to_string(i) + " ", mw = where + "mixer.";
      LayerSpec s;
      const JVal* ty = L.get("type");
      const JVal* mx = L.get("mixer");
      if (!ty || ty->type != JVal::Str) { *err = "config: " + where + "type"; return false; }
      if (!mx || mx->type != JVal::Obj) { *err = "config: " + where + "mixer"; return false; }
      if (!whole(mx, "heads", 1, &s.heads, mw) || !whole(mx, "vdim", 1, &s.vdim, mw)) return false;
      if (ty->str == "latent_attention") {
        s.kind = MIX_LATENT;
        if (!whole(mx, "dim", 1, &s.dim, mw) || !whole(mx, "rot_dim", 0, &s.rot_dim, mw) || !whole(mx, "kv_rank", 1, &s.kv_rank, mw)) return false;
        if (given(mx, "q_rank") && !whole(mx, "q_rank", 1, &s.q_rank, mw)) return false;    // otherwise the checkpoint says it
        s.rot_dims = s.rot_dim / 2 * 2;
        if (const JVal* rot = mx->get("rot")) {
          if (rot->type == JVal::Obj) {
            if (given(rot, "dims") && !whole(rot, "dims", 0, &s.rot_dims, mw + "rot.")) return false;
            if (jnum(rot, "base", &d)) s.rot_base = d;
          }
        }
        if (s.rot_dims > s.rot_dim || s.rot_dims % 2 || !(s.rot_base > 0)) { *err = "config: " + mw + "rot"; return false; }
        s.scale = 1.0f / sqrtf(static_cast<float>(s.dim + s.rot_dim));
        if (jnum(mx, "scale", &d)) s.scale = static_cast<float>(d);
        if (given(mx, "kv_from")) {
          if (!whole(mx, "kv_from", 0, &s.kv_from, mw)) return false;
          const LayerSpec* src = s.kv_from < static_cast<int>(i) ? &spec[s.kv_from] : nullptr;
          if (!src || !src->own_cache()) { *err = "config: " + mw + "kv_from names no earlier attention layer with a cache of its own"; return false; }
          if (src->kv_rank != s.kv_rank || src->rot_dim != s.rot_dim || src->rot_dims != s.rot_dims || src->rot_base != s.rot_base) {
            *err = "config: " + mw + "kv_from: kv_rank, rot_dim and rotation differ from that layer's";
            return false;
          }
        }
      } else if (ty->str == "hgrn2") {
        s.kind = MIX_HGRN2;
        if (!whole(mx, "dim", 1, &s.dim, mw)) return false;
      } else if (ty->str == "mamba2") {
        s.kind = MIX_MAMBA2;
        if (!whole(mx, "state", 1, &s.dim, mw)) return false;
        if (given(mx, "groups") && !whole(mx, "groups", 1, &s.groups, mw)) return false;
        if (given(mx, "norm_groups") && !whole(mx, "norm_groups", 1, &s.norm_groups, mw)) return false;
        if (given(mx, "conv") && !whole(mx, "conv", 1, &s.taps, mw)) return false;
        if (s.heads % s.groups) { *err = "config: " + mw + "heads is no multiple of groups"; return false; }
        if ((static_cast<long long>(s.heads) * s.vdim) % s.norm_groups) { *err = "config: " + mw + "norm_groups does not divide heads * vdim"; return false; }
        if (static_cast<long long>(s.heads) * s.vdim / s.norm_groups > 12000) { *err = "config: " + mw + "a norm group above 12000 channels"; return false; }
      } else { *err = "config: unknown mixer \"" + ty->str + "\""; return false; }
      if (s.kind != MIX_LATENT && s.dim > 1024) { *err = "config: " + where + "a recurrent state of more than 1024 rows"; return false; }
      const JVal* mlp = L.get("mlp");
      if (mlp && mlp->type == JVal::Obj) {
        const JVal* kind = mlp->get("kind");
        if (!kind || kind->type != JVal::Str || kind->str != "dense") { *err = "config: " + where + "mlp.kind (dense)"; return false; }
        s.mlp = true;
        if (given(mlp, "ff") && !whole(mlp, "ff", 1, &s.ff, where + "mlp.")) return false;   // otherwise the checkpoint says it
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
    const int HD = s.heads * s.dim, HV = s.heads * s.vdim;
    s.k_out = HV;
    if (s.kind == MIX_LATENT) {
      block(&s.off_dq, s.q_rank);
      if (s.own_cache()) block(&s.off_dkv, s.kv_rank + s.rot_dim);
      block(&s.off_g, s.heads);
    } else if (s.kind == MIX_HGRN2) {
      block(&s.off_q, HD);
      block(&s.off_f, HD);
      block(&s.off_v, HV);
      s.rec_floats = static_cast<size_t>(HD) * s.vdim;
    } else {
      s.conv_c = HV + 2 * s.groups * s.dim;
      block(&s.off_z, HV);
      block(&s.off_xbc, s.conv_c);      // x, B, C: one run of convolved channels
      block(&s.off_dt, s.heads);
      s.conv_floats = static_cast<size_t>(s.taps - 1) * s.conv_c;
      s.rec_floats = static_cast<size_t>(HD) * s.vdim;
    }
    s.n_in = at;
    // a wide row is filled up to whole 256-row weight tiles (rows of zeros nobody reads), which the fused GEMM form asks for
    const int full = (at + 255) / 256 * 256;
    if (at >= 1024 && full - at <= at / 8) s.n_in = full;
  }

  int inspect(const CheckpointReader& ck, std::string* err) override {
    std::vector<int64_t> sh;
    for (size_t i = 0; i < spec.size(); ++i) {
      LayerSpec& s = spec[i];
      const std::string p = "l" + std::to_string(i) + ".";
      if (s.kind == MIX_LATENT && s.q_rank == 0) {
        if (!ck.shape(p + "mix.dq", &sh) || sh.size() != 2) { *err = p + "mix.dq"; return -4; }
        s.q_rank = static_cast<int>(sh[0]);
      }
      if (s.mlp && s.ff == 0) {
        if (!ck.shape(p + "mlp.up", &sh) || sh.size() != 2) { *err = p + "mlp.up"; return -4; }
        s.ff = static_cast<int>(sh[0]);
      }
      layout(s);
    }
    return 0;
  }

  template <typename P>
  int dalloc(P** p, size_t bytes) {
    void* q = nullptr;
    if (cudaMalloc(&q, std::max<size_t>(bytes, 16)) != cudaSuccess) { set_error("Soselix: device allocation of %zu bytes failed", bytes); return -3; }
    cudaMemsetAsync(q, 0, std::max<size_t>(bytes, 16), env.stream);
    allocs.push_back(q);
    *p = static_cast<P*>(q);
    return 0;
  }

  int init(const ModelEnv& e) override {
    env = e;
    const size_t es = dtype_bytes(dt);
    wts.resize(spec.size());
    int max_in = 8, max_out = 8, max_cq = 8, max_q = 8, max_ql = 0, max_ol = 0, max_xc = 0, max_rec = 0, max_ff = 0;
    for (size_t i = 0; i < spec.size(); ++i) {
      const LayerSpec& s = spec[i];
      if ((s.kind == MIX_LATENT && s.q_rank < 1) || (s.mlp && s.ff < 1)) { set_error("Soselix: layer %d: q_rank or mlp.ff is not known", static_cast<int>(i)); return -1; }
      max_in = std::max(max_in, s.n_in); max_out = std::max(max_out, s.k_out); max_ff = std::max(max_ff, s.ff);
      if (s.kind == MIX_LATENT) {
        max_cq = std::max(max_cq, s.q_rank); max_q = std::max(max_q, s.heads * (s.dim + s.rot_dim));
        max_ql = std::max(max_ql, s.heads * (s.kv_rank + s.rot_dim)); max_ol = std::max(max_ol, s.heads * s.kv_rank);
      } else {
        max_rec = std::max(max_rec, s.k_out); max_xc = std::max(max_xc, s.conv_c);
      }
    }
    int rc = 0;
    auto mat = [&](void** p, size_t rows, size_t cols) { return dalloc(p, rows * cols * es); };
    auto vec = [&](float** p, size_t n) { return dalloc(p, n * sizeof(float)); };
    rc |= mat(&embed, V, W) | mat(&head, V, W) | vec(&fin_w, W);
    for (size_t i = 0; i < spec.size() && !rc; ++i) {
      const LayerSpec& s = spec[i];
      if (s.own_cache()) rc |= dalloc(&run[i].cache, static_cast<size_t>(e.num_blocks) * e.page * (s.kv_rank + s.rot_dim) * es);
      if (s.kind != MIX_LATENT)
        rc |= dalloc(&run[i].conv, static_cast<size_t>(e.num_slots) * s.conv_floats * sizeof(float)) |
              dalloc(&run[i].state, static_cast<size_t>(e.num_slots) * s.rec_floats * sizeof(float));
    }
    for (size_t i = 0; i < spec.size() && !rc; ++i) {
      const LayerSpec& s = spec[i];
      LayerWeights& w = wts[i];
      if (s.kv_from >= 0) run[i].cache = run[s.kv_from].cache;   // the same pages, written by that layer
      const int HD = s.heads * s.dim;
      rc |= mat(&w.w_in, s.n_in, W) | mat(&w.w_out, W, s.k_out) | vec(&w.norm1, W);
      if (s.kind == MIX_LATENT) {
        rc |= mat(&w.w_uq, static_cast<size_t>(s.heads) * (s.dim + s.rot_dim), s.q_rank) | mat(&w.uk_t, static_cast<size_t>(s.heads) * s.kv_rank, s.dim) |
              mat(&w.w_uv, s.k_out, s.kv_rank) | vec(&w.cq_norm, s.q_rank) | vec(&w.sink, s.heads);
        if (s.own_cache()) rc |= vec(&w.c_norm, s.kv_rank);
        if (s.kv_from >= 0) w.rope = wts[s.kv_from].rope;
        else {
          rc |= dalloc(&w.rope, static_cast<size_t>(e.max_model_len) * std::max(1, s.rot_dims / 2) * sizeof(float2));
          if (!rc && rope_table_interleaved(w.rope, e.max_model_len, s.rot_dims, s.rot_base, e.stream)) rc = -2;
        }
      } else if (s.kind == MIX_HGRN2) {
        rc |= vec(&w.f_b, HD) | vec(&w.lower, HD) | vec(&w.o_norm, s.vdim);
      } else {
        rc |= vec(&w.conv_w, static_cast<size_t>(s.conv_c) * s.taps) | vec(&w.conv_b, s.conv_c) | vec(&w.dt_b, s.heads) | vec(&w.dt_rate, s.heads) |
              vec(&w.skip, s.heads) | vec(&w.o_norm, s.k_out);
      }
      if (s.mlp) rc |= vec(&w.norm2, W) | mat(&w.w_up, s.ff, W) | mat(&w.w_down, W, s.ff) | vec(&w.up_b, s.ff) | vec(&w.down_b, W);
    }
    if (rc) return rc;
    const size_t T = e.Tcap;
    row_cap = static_cast<int>(std::min<size_t>(T, 256));
    rc |= vec(&x, T * W) | mat(&h, T, W) | mat(&inb, T, max_in) | mat(&yb, T, max_out) | mat(&ao, T, W) | mat(&hrow, row_cap, W) |
          vec(&logits, static_cast<size_t>(row_cap) * V);
    if (max_ql) rc |= mat(&cq, T, max_cq) | mat(&qb, T, max_q) | vec(&qlat, T * max_ql) | vec(&olat, T * max_ol);
    if (max_rec) rc |= vec(&o32, T * max_rec);
    if (max_xc) rc |= mat(&xc, T, max_xc);
    if (max_ff) rc |= mat(&hid, T, max_ff) | mat(&fo, T, W);
    if (max_ol && dt == DT_BF16) {
      split_ws_floats = 1024ll * (max_ol + 2 * 64);   // rows x splits <= 1024 of [kv_rank + 2] per head
      rc |= vec(&split_ws, split_ws_floats);
    }
    if (rc) return rc;
    register_tensors();
    rc = setup_tc();
    if (rc) return rc;
    return cudaStreamSynchronize(e.stream) == cudaSuccess ? 0 : -2;
  }

  // The projections of a bf16 model run on the tcgen05 pair GEMM (gemm2_tcgen05.cu) where their shapes allow it (rows and
  // columns in multiples of 8): input, query, output, up and down projection.  The per-head products of the latent attention
  // (fp32 on one side) and every projection of an fp32 model stay on linear.cu.  B200_SX_TC=0 keeps everything there (A/B
  // knob).
  int setup_tc() {
    const char* ev = getenv("B200_SX_TC");
    use_tc = dt == DT_BF16 && !(ev && atoi(ev) == 0) && W % 8 == 0 && gemm_variant() == 2;
    if (!use_tc) return 0;
    int maxN = W;
    for (auto& s : spec) maxN = std::max(std::max(maxN, s.n_in), std::max(s.ff, s.kind == MIX_LATENT ? s.heads * (s.dim + s.rot_dim) : 0));
    const size_t ws_bytes = std::max(gemm_workspace_bytes(env.sms), gemm_deferred_ws_bytes(env.sms));
    if (dalloc(&gemm_ws, ws_bytes)) return -3;
    const size_t n_counters = 2ull * (maxN / 128 + 2) * (env.Tcap / 32 + 2);
    if (dalloc(&gemm_counters, n_counters * sizeof(int)) || dalloc(&gemm_flags, static_cast<size_t>(env.sms) * 2 * sizeof(int))) return -3;
    if (const char* e = getenv("B200_SX_FUSE")) fuse = atoi(e) != 0;              // A/B knobs
    if (const char* e = getenv("B200_SX_FEW_ROWS")) few_rows = atoi(e);
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
    if (!maps(xm_h, h, W)) { use_tc = false; return 0; }
    for (size_t i = 0; i < spec.size(); ++i) {
      const LayerSpec& s = spec[i];
      LayerWeights& w = wts[i];
      w.tc_in = plan(&w.p_in, w.w_in, s.n_in, W);
      w.tc_out = plan(&w.p_out, w.w_out, W, s.k_out) && maps(w.xm_out, yb, s.k_out);
      if (s.kind == MIX_LATENT) w.tc_uq = plan(&w.p_uq, w.w_uq, s.heads * (s.dim + s.rot_dim), s.q_rank) && maps(w.xm_cq, cq, s.q_rank);
      if (s.mlp) {
        w.tc_up = plan(&w.p_up, w.w_up, s.ff, W);
        w.tc_down = plan(&w.p_down, w.w_down, W, s.ff) && maps(w.xm_hid, hid, s.ff);
      }
    }
    return 0;
  }

  void reg(const std::string& name, void* p, size_t bytes) { tensors[name] = {p, bytes}; }
  void register_tensors() {
    const size_t es = dtype_bytes(dt);
    reg("embed", embed, static_cast<size_t>(V) * W * es);
    reg("head", head, static_cast<size_t>(V) * W * es);
    for (size_t i = 0; i < spec.size(); ++i) reg("l" + std::to_string(i) + ".w_in", wts[i].w_in, static_cast<size_t>(spec[i].n_in) * W * es);
  }

  // ------------------------------------------------------------ weights
  // host fp32 [rows, cols] -> device rows [row0, row0 + rows) of a matrix with `cols` columns
  int put(void* dst, size_t row0, const float* src, size_t rows, size_t cols) {
    const size_t es = dtype_bytes(dt);
    std::vector<uint8_t> tmp(rows * cols * es);
    if (dt == DT_F32) memcpy(tmp.data(), src, tmp.size());
    else {
      bf16* o = reinterpret_cast<bf16*>(tmp.data());
      for (size_t i = 0; i < rows * cols; ++i) o[i] = __float2bfloat16_rn(src[i]);
    }
    return cudaMemcpy(static_cast<uint8_t*>(dst) + row0 * cols * es, tmp.data(), tmp.size(), cudaMemcpyHostToDevice) == cudaSuccess ? 0 : -2;
  }
  int putf(float* dst, const std::vector<float>& src) {
    return cudaMemcpy(dst, src.data(), src.size() * sizeof(float), cudaMemcpyHostToDevice) == cudaSuccess ? 0 : -2;
  }
  static float softplus(float v) { return static_cast<float>(v > 0.f ? v + log1p(exp(-static_cast<double>(v))) : log1p(exp(static_cast<double>(v)))); }

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
#define MAT(name, dst, row0, rows, cols) do { if (!get(name, rows, cols)) return -4; rc |= put(dst, row0, v.data(), rows, cols); } while (0)
#define VEC(name, dst, n) do { if (!get(name, 1, n)) return -4; rc |= putf(dst, v); } while (0)
#define NORM1(name, dst) do { if (!get(name, 1, 1)) return -4; const float g_ = v[0]; v.assign(W, g_); rc |= putf(dst, v); } while (0)   // one number, spread over the width
    MAT("embed", embed, 0, V, W);
    MAT("head", head, 0, V, W);
    NORM1("final.norm", fin_w);
    for (size_t i = 0; i < spec.size(); ++i) {
      const LayerSpec& s = spec[i];
      LayerWeights& w = wts[i];
      const std::string p = "l" + std::to_string(i) + ".", mx = p + "mix.", f = p + "mlp.";
      const int HD = s.heads * s.dim, HV = s.heads * s.vdim;
      NORM1(p + "norm1", w.norm1);
      if (s.kind == MIX_LATENT) {
        const int C = s.kv_rank, D = s.dim;
        MAT(mx + "dq", w.w_in, s.off_dq, s.q_rank, W);
        VEC(mx + "dq.norm", w.cq_norm, s.q_rank);
        MAT(mx + "uq", w.w_uq, 0, s.heads * (D + s.rot_dim), s.q_rank);
        if (s.own_cache()) {
          MAT(mx + "dkv", w.w_in, s.off_dkv, C + s.rot_dim, W);
          VEC(mx + "dkv.norm", w.c_norm, C);
        }
        if (!get(mx + "uk", HD, C)) return -4;
        std::vector<float> t(static_cast<size_t>(HD) * C);     // per head transposed: the latent query projection
        for (int hd = 0; hd < s.heads; ++hd)
          for (int r = 0; r < D; ++r)
            for (int k = 0; k < C; ++k) t[(static_cast<size_t>(hd) * C + k) * D + r] = v[(static_cast<size_t>(hd) * D + r) * C + k];
        rc |= put(w.uk_t, 0, t.data(), static_cast<size_t>(s.heads) * C, D);
        MAT(mx + "uv", w.w_uv, 0, HV, C);
        VEC(mx + "sink", w.sink, s.heads);
        MAT(mx + "g", w.w_in, s.off_g, s.heads, W);
      } else if (s.kind == MIX_HGRN2) {
        MAT(mx + "q", w.w_in, s.off_q, HD, W);
        MAT(mx + "f", w.w_in, s.off_f, HD, W);
        VEC(mx + "f.b", w.f_b, HD);
        VEC(mx + "lower", w.lower, HD);
        MAT(mx + "v", w.w_in, s.off_v, HV, W);
        VEC(mx + "norm", w.o_norm, s.vdim);
      } else {
        if (!get(mx + "in", HV + s.conv_c + s.heads, W)) return -4;
        rc |= put(w.w_in, s.off_z, v.data(), HV, W) | put(w.w_in, s.off_xbc, v.data() + static_cast<size_t>(HV) * W, s.conv_c, W) |
              put(w.w_in, s.off_dt, v.data() + static_cast<size_t>(HV + s.conv_c) * W, s.heads, W);
        if (!get(mx + "conv", s.conv_c, s.taps)) return -4;
        rc |= putf(w.conv_w, v);
        VEC(mx + "conv.b", w.conv_b, s.conv_c);
        VEC(mx + "dt_bias", w.dt_b, s.heads);
        if (!get(mx + "A_log", 1, s.heads)) return -4;
        for (auto& a : v) a = static_cast<float>(-exp(static_cast<double>(a)));     // the decay's rate, once
        rc |= putf(w.dt_rate, v);
        VEC(mx + "D", w.skip, s.heads);
        VEC(mx + "norm", w.o_norm, HV);
      }
      MAT(mx + "o", w.w_out, 0, W, HV);
      if (!s.mlp) continue;
      NORM1(p + "norm2", w.norm2);
      MAT(f + "up", w.w_up, 0, s.ff, W);
      VEC(f + "up.b", w.up_b, s.ff);
      MAT(f + "down", w.w_down, 0, W, s.ff);
      VEC(f + "down.b", w.down_b, W);
      if (!get(f + "act", 1, 2)) return -4;
      w.act_pos = softplus(v[0]);
      w.act_neg = 0.5f + softplus(v[1]);
    }
#undef MAT
#undef VEC
#undef NORM1
    if (rc) { *err = "copying weights to the device failed"; return -2; }
    return 0;
  }

  // Seeded random weights of a plausible scale (benchmarks: there is no checkpoint of a real size).
  int randomize(uint64_t seed) override {
    cudaStream_t st = env.stream;
    int rc = 0;
    uint64_t k = seed * 1000003ull + 57;
    auto M = [&](void* p, size_t n, float sc) { if (p) rc |= fill_uniform(p, dt, n, ++k, sc, 0.f, st); };
    auto F = [&](float* p, size_t n, float sc, float off) { if (p) rc |= fill_uniform(p, DT_F32, n, ++k, sc, off, st); };
    auto by = [](int n) { return 1.7f / sqrtf(static_cast<float>(n)); };
    M(embed, static_cast<size_t>(V) * W, 1.f);
    M(head, static_cast<size_t>(V) * W, by(W));
    F(fin_w, W, 0.f, 1.f);
    for (size_t i = 0; i < spec.size(); ++i) {
      const LayerSpec& s = spec[i];
      LayerWeights& w = wts[i];
      const size_t HD = static_cast<size_t>(s.heads) * s.dim;
      M(w.w_in, static_cast<size_t>(s.n_in) * W, by(W));
      M(w.w_out, static_cast<size_t>(W) * s.k_out, by(s.k_out));
      F(w.norm1, W, 0.f, 1.f);
      if (s.kind == MIX_LATENT) {
        M(w.w_uq, static_cast<size_t>(s.heads) * (s.dim + s.rot_dim) * s.q_rank, by(s.q_rank));
        M(w.uk_t, HD * s.kv_rank, by(s.kv_rank));
        M(w.w_uv, static_cast<size_t>(s.k_out) * s.kv_rank, by(s.kv_rank));
        F(w.cq_norm, s.q_rank, 0.1f, 1.f); F(w.c_norm, s.kv_rank, 0.1f, 1.f); F(w.sink, s.heads, 1.f, 0.f);
      } else if (s.kind == MIX_HGRN2) {
        F(w.f_b, HD, 1.f, 2.f); F(w.lower, HD, 0.45f, 0.45f); F(w.o_norm, s.vdim, 0.1f, 1.f);
      } else {
        F(w.conv_w, static_cast<size_t>(s.conv_c) * s.taps, 0.5f, 0.3f); F(w.conv_b, s.conv_c, 0.1f, 0.f);
        F(w.dt_b, s.heads, 1.f, -3.f); F(w.dt_rate, s.heads, 0.4f, -0.5f); F(w.skip, s.heads, 0.2f, 1.f); F(w.o_norm, s.k_out, 0.1f, 1.f);
      }
      if (!s.mlp) continue;
      F(w.norm2, W, 0.f, 1.f);
      M(w.w_up, static_cast<size_t>(s.ff) * W, by(W)); F(w.up_b, s.ff, 0.1f, 0.f);
      M(w.w_down, static_cast<size_t>(W) * s.ff, by(s.ff)); F(w.down_b, W, 0.1f, 0.f);
      w.act_pos = 0.8f; w.act_neg = 1.2f;
    }
    if (rc) return -2;
    return cudaStreamSynchronize(st) == cudaSuccess ? 0 : -2;
  }

  // ------------------------------------------------------------ forward
  // Y = X W^T, with bias and xIELU behind it where the epilogue is given.  Steps of up to 16 tokens stream the weights through
  // linear.cu's fragment kernel.  Larger steps take the pair GEMM; in its fused form (whole 256-row tiles, at least one tile
  // per CTA pair) every tile leaves through the epilogue, otherwise the epilogue is a pass of its own over the result.
  struct Epilogue {
    const float* bias = nullptr;
    float a_pos = 0.f, a_neg = 0.f;
  };
  int project(const GemmPlan& plan, bool tc, const CUtensorMap* xm, const void* X, const void* Wm, void* Y, int T, int N, int K, const Epilogue* ep = nullptr) {
    if (tc && T > few_rows) {
      const int bn = block_n(plan, T);
      if (fuse && N % 256 == 0 && T > 128 && N / 256 * ((T + bn - 1) / bn) >= plan.max_ctas / 2) {
        Gemm2Epi e;
        memset(&e, 0, sizeof(e));
        e.epi = ep ? GEMM3_EPI_BIAS_XIELU : GEMM3_EPI_PLAIN;
        e.out = static_cast<bf16*>(Y); e.ldo = N;
        e.flags = gemm_flags; e.epoch = ++gemm_epoch;
        if (ep) { e.bias = ep->bias; e.a_pos = ep->a_pos; e.a_neg = ep->a_neg; }
        return gemm2_run_fused(plan, xm[gemm_block_n_index(bn)], bn, T, e, env.stream);
      }
      const int rc = gemm_run(plan, xm[gemm_block_n_index(bn)], bn, Y, N, T, env.stream);
      return rc || !ep ? rc : bias_act(Y, N, ep->bias, LIN_XIELU, dt, T, N, env.stream, ep->a_pos, ep->a_neg);
    }
    LinearArgs la = linear_args(X, dt, Wm, dt, Y, dt, T, N, K);
    if (ep) { la.bias = ep->bias; la.act = LIN_XIELU; la.a_pos = ep->a_pos; la.a_neg = ep->a_neg; }
    return linear(la, env.stream);
  }
  // Token-tile size: where 512-token tiles neither fill the pairs nor are close enough to one whole tile per pair (that form
  // takes up to 64 k-blocks), 256-token tiles give the fused form its tile per pair.
  int block_n(const GemmPlan& p, int T) const {
    const int bn = gemm_block_n_for(T), pairs = p.max_ctas / 2;
    if (bn != 512 || !fuse || p.N % 256) return bn;
    const int t512 = p.N / 256 * ((T + 511) / 512), t256 = p.N / 256 * ((T + 255) / 256);
    const bool whole = p.K <= 4096 && t512 * 5 >= pairs * 3;
    return t512 < pairs && !whole && t256 >= pairs ? 256 : bn;
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

  // the write-back of the last sublayer, still to be applied by the next boundary
  struct Pending {
    const void* y = nullptr;
    const float* bias = nullptr;
  };
  SandwichArgs boundary(const Pending& p, const float* norm_w, void* out, const int* row_index, int rows) {
    SandwichArgs a;
    a.x = x; a.y = p.y; a.ty = dt; a.y_bias = p.bias; a.mult = mult;
    a.post_w = nullptr; a.pre_w = norm_w; a.eps = eps;
    a.h = out; a.th = dt; a.row_index = row_index; a.rows = rows; a.W = W;
    return a;
  }

  int mix_latent(const LayerSpec& s, const LayerWeights& w, const LayerRun& r, const StepBatch& b, int64_t& nl) {
    cudaStream_t st = env.stream;
    const int T = b.T, C = s.kv_rank, R = s.rot_dim, E = C + R, Q = s.heads * (s.dim + R);
    int rc = 0;
    // norm of the query latent; the token's cache row, where this layer makes its own
    LatentPrepArgs p = {};
    p.t = dt; p.eps = eps; p.rope = w.rope; p.rot_dims = s.rot_dims; p.half_pairs = true; p.positions = b.pos; p.slots = b.slots;
    p.cache = r.cache; p.qlat = qlat; p.T = T; p.heads = s.heads; p.dim = s.dim; p.rot_dim = R; p.kv_rank = C;
    LatentPrepArgs pq = p;
    if (s.own_cache()) { p.dkv = col(inb, s.off_dkv); p.lddkv = s.n_in; p.norm_w = w.c_norm; }
    p.cq = col(inb, s.off_dq); p.ldcq = s.n_in; p.cq_w = w.cq_norm; p.q_rank = s.q_rank; p.cq_out = cq; p.ldcq_out = s.q_rank;
    KRN("latent_prep", latent_prep(p, st));
    KRN("proj_q", project(w.p_uq, w.tc_uq, w.xm_cq, cq, w.w_uq, qb, T, Q, s.q_rank));
    if (R > 0) {
      pq.q = qb; pq.ldq = Q;
      KRN("latent_q_rotate", latent_prep(pq, st));
    }
    // latent query: per head [T, dim] x [kv_rank, dim]^T into the head's first kv_rank columns of qlat
    LinearArgs lq = linear_args(qb, dt, w.uk_t, dt, qlat, DT_F32, T, C, s.dim);
    lq.ldx = Q; lq.ldy = s.heads * E; lq.batch = s.heads; lq.xbs = s.dim + R; lq.wbs = static_cast<long long>(C) * s.dim; lq.ybs = E;
    KRN("latent_q_absorb", linear(lq, st));
    LatentAttnArgs a = {};
    a.qlat = qlat; a.cache = r.cache; a.t = dt; a.positions = b.pos; a.seq_of_tok = b.seq_of_tok; a.block_tables = b.btab;
    a.max_blocks = b.max_blocks; a.page = env.page; a.olat = olat;
    a.T = T; a.heads = s.heads; a.kv_rank = C; a.rot_dim = R; a.window = env.max_model_len; a.scale = s.scale;
    a.seqs = b.seqs; a.nseq = b.nseq; a.max_ctx = b.max_ctx; a.split_ws = split_ws; a.split_ws_floats = split_ws_floats;
    a.sink = w.sink; a.gate = col(inb, s.off_g); a.ldg = s.n_in;
    KRN("latent_attention", latent_attention(a, st));
    // values: per head [T, kv_rank] x [vdim, kv_rank]^T into the head's columns of the output projection's input
    LinearArgs lv = linear_args(olat, DT_F32, w.w_uv, dt, yb, dt, T, s.vdim, C);
    lv.ldx = s.heads * C; lv.ldy = s.k_out; lv.batch = s.heads; lv.xbs = C; lv.wbs = static_cast<long long>(s.vdim) * C; lv.ybs = s.vdim;
    KRN("latent_v_expand", linear(lv, st));
    return rc;
  }

  GlaArgs scan_args(const LayerSpec& s, const LayerRun& r, const StepBatch& b) {
    GlaArgs g = {};
    g.t = dt; g.inv_tau = 1.f; g.q_scale = 1.f; g.T = b.T;
    g.states = r.state; g.seqs = b.seqs; g.nseq = b.nseq;
    g.heads = s.heads; g.dim = s.dim; g.vdim = s.vdim; g.o = o32;
    return g;
  }

  int mix_hgrn2(const LayerSpec& s, const LayerWeights& w, const LayerRun& r, const StepBatch& b, int64_t& nl) {
    cudaStream_t st = env.stream;
    int rc = 0;
    GlaArgs g = scan_args(s, r, b);
    g.qkv = inb; g.ld = s.n_in; g.q_off = s.off_q; g.k_off = s.off_f; g.v_off = s.off_v;
    g.act = GLA_ACT_SILU_Q; g.z_bias = w.f_b; g.fgate_lower = w.lower;
    KRN("hgrn2_scan", gla_scan(g, st));
    OutGateArgs og = {};
    og.o = o32; og.w = w.o_norm; og.eps = eps;
    og.y = yb; og.ldy = s.k_out; og.t = dt; og.T = b.T; og.heads = s.heads; og.vdim = s.vdim;
    og.joint = false; og.gate_act = GATE_SILU; og.out_scale = 1.f;
    KRN("hgrn2_out_norm", recurrent_out_gate(og, st));
    return rc;
  }

  int mix_mamba2(const LayerSpec& s, const LayerWeights& w, const LayerRun& r, const StepBatch& b, int64_t& nl) {
    cudaStream_t st = env.stream;
    const int HV = s.k_out;
    int rc = 0;
    ShortConvArgs cc = {};
    cc.u = col(inb, s.off_xbc); cc.ldu = s.n_in; cc.t = dt; cc.w = w.conv_w; cc.bias = w.conv_b; cc.act = CONV_SILU;
    cc.y = xc; cc.ldy = s.conv_c; cc.ty = dt; cc.state = r.conv;
    cc.seq_of_tok = b.seq_of_tok; cc.seqs = b.seqs; cc.nseq = b.nseq; cc.T = b.T; cc.C = s.conv_c; cc.taps = s.taps;
    KRN("short_conv", short_conv(cc, st));
    if (s.taps > 1) KRN("conv_carry", short_conv_carry(cc, st));
    GlaArgs g = scan_args(s, r, b);
    g.qkv = xc; g.ld = s.conv_c; g.v_off = 0; g.k_off = HV; g.q_off = HV + s.groups * s.dim;
    g.group = s.heads / s.groups;
    g.dt_pre = col(inb, s.off_dt); g.ld_dt = s.n_in; g.dt_bias = w.dt_b; g.dt_rate = w.dt_rate;
    KRN("mamba2_scan", gla_scan(g, st));
    GatedGroupNormArgs gn = {};
    gn.o = o32; gn.x = xc; gn.ldx = s.conv_c; gn.skip = w.skip; gn.z = col(inb, s.off_z); gn.ldz = s.n_in; gn.w = w.o_norm; gn.eps = eps;
    gn.y = yb; gn.ldy = HV; gn.t = dt; gn.T = b.T; gn.heads = s.heads; gn.vdim = s.vdim; gn.groups = s.norm_groups;
    KRN("mamba2_gate_norm", gated_group_norm(gn, st));
    return rc;
  }

  int forward(const StepBatch& b, int* sampled, float* host_logits, int64_t* launches) override {
    cudaStream_t st = env.stream;
    const int T = b.T;
    int rc = 0;
    int64_t nl = 0;
    KRN("embed", embed_scaled(embed, dt, b.ids, x, T, W, V, embed_scale, 1, 0, st));
    Pending pend;
    for (size_t li = 0; li < spec.size() && !rc; ++li) {
      const LayerSpec& s = spec[li];
      const LayerWeights& w = wts[li];
      const LayerRun& r = run[li];
      KRN("residual_norm", sandwich_step(boundary(pend, w.norm1, h, nullptr, T), st));
      KRN("proj_in", project(w.p_in, w.tc_in, xm_h, h, w.w_in, inb, T, s.n_in, W));
      if (s.kind == MIX_LATENT) rc |= mix_latent(s, w, r, b, nl);
      else if (s.kind == MIX_HGRN2) rc |= mix_hgrn2(s, w, r, b, nl);
      else rc |= mix_mamba2(s, w, r, b, nl);
      KRN("proj_out", project(w.p_out, w.tc_out, w.xm_out, yb, w.w_out, ao, T, W, s.k_out));
      pend.y = ao; pend.bias = nullptr;
      if (s.mlp) {
        KRN("residual_norm", sandwich_step(boundary(pend, w.norm2, h, nullptr, T), st));
        Epilogue ep;
        ep.bias = w.up_b; ep.a_pos = w.act_pos; ep.a_neg = w.act_neg;
        KRN("ff_up", project(w.p_up, w.tc_up, xm_h, h, w.w_up, hid, T, s.ff, W, &ep));
        KRN("ff_down", project(w.p_down, w.tc_down, w.xm_hid, hid, w.w_down, fo, T, W, s.ff));
        pend.y = fo; pend.bias = w.down_b;
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
    if (rc) { set_error("Soselix forward: %s failed with %d (%s)", failed_kernel, failed_rc, cudaGetErrorString(cudaGetLastError())); return -2; }
    return 0;
  }
};

}  // namespace

#undef KRN

std::unique_ptr<Model> make_soselix(const JVal& config, DType dtype, std::string* err) {
  std::unique_ptr<Soselix> m(new Soselix(dtype));
  if (!m->parse(config, err)) return nullptr;
  return std::unique_ptr<Model>(m.release());
}

}  // namespace b200
