// kalesun_model.cu — the Kalesun architecture on the runner's model interface (model.hpp).
//
// Kalesun is a decoder-only model on an f32 residual stream that is normed AFTER every sum,
//     x <- rms(alpha x + mixer(x)) w1;   x <- rms(alpha x + ff(x)) w2        (a layer may have no feed-forward),
// so every sublayer reads the stream itself (in the operand type).  Plain embedding, a final RMS norm and a tied output head.
// Three kinds of mixer, in any order:
//   "attention"  grouped-query softmax attention over the paged cache (capped_attn.cu): a weighted RMS norm per query and key
//                head, then rotary on the first rot.dims values (value i paired with i + dims / 2; frequencies optionally
//                scaled by wavelength); a sliding window that keeps the sequence's first keys; a learned sink per head; one
//                sigmoid gate per head.  Layers with v_mix blend their values with those of the FIRST such layer (same token,
//                same step) before they are cached.
//   "delta"      the gated delta rule with one decay per head (recurrence.cu): q, k, v through a short causal convolution and
//                SiLU, q and k made unit vectors, beta = sigmoid; per-head RMS norm with a shared weight and a SiLU gate.
//   "gla"        gated linear attention with a decay per key channel, sigmoid(A2 A1 x + b)^(1 / tau) (recurrence.cu); the
//                same output norm and gate.
// The recurrent mixers' state matrices and the convolutions' last inputs live in per-sequence state slots that the
// scheduler hands out.  Feed-forward: dense with the clamped gate (g' sigmoid(1.702 g') (u' + 1)), or a mixture of such
// experts routed on the logits (the `top` largest of W_r x + b, softmax over the chosen alone).
//
// bf16 engines: weights, projections' operands, sublayer outputs, q and the cache in bf16 with f32 accumulation; the residual,
// norms, scores, softmax, rotary angles, router, convolutions, decays, recurrences and the low-rank decay product in f32.
// f32 engines: everything in f32.
//
// config.json keys: vocab, width, norm.eps, postln_alpha, layers[] of {type, mixer, mlp}.  layers[i].mixer by type:
// attention: heads, kv_heads, dim, vdim, scale, mask.{size,keep_first}, rot.{base,dims,scaling.{factor,low,high,original}}, v_mix;
// delta: heads, kv_heads, dim, vdim, conv;  gla: heads, dim, vdim, tau, low_rank (synthetic weights only).
// layers[i].mlp: null | {kind "dense", ff, limit} | {kind "moe", expert.{ff,limit}, router.{experts,top}}.
// tensors: embed, final.norm, l<i>.norm{1,2}, l<i>.mix.{q,k,v,g,o}, l<i>.mix.{q.norm,k.norm,sink,vmix} (attention),
// l<i>.mix.{q,k,v}.conv, l<i>.mix.{a,b,A_log,dt_bias,norm} (delta), l<i>.mix.{a1,a2,a2.b,norm} (gla), l<i>.mlp.{gate,up,down}
// (dense), l<i>.mlp.{router,router.b}, l<i>.mlp.e<k>.{gate,up,down} (experts).
#include <algorithm>
#include <array>
#include <map>

#include "model_base.hpp"

namespace nvllm {
namespace {

#define RUN(expr)                   \
  do {                              \
    int _rc = (expr);               \
    if (_rc != 0) return _rc;       \
  } while (0)

enum MixKind { kAttention = 0, kDelta = 1, kGla = 2 };
enum FfKind { kNone = 0, kDense = 1, kExperts = 2 };

struct Layer {
  int mix = kAttention, ffk = kNone;
  int H = 0, G = 0, D = 0, V = 0;
  // attention
  float scale = 1.f;
  int window = 0, keep_first = 0, rot_dims = 0;
  double rot_base = 10000.0;
  std::array<double, 4> rot_scaling{0.0, 1.0, 2.0, 1.0};   // factor (0: none), low, high, original
  bool v_mix = false, v_source = false;                     // v_source: the first layer with v_mix, whose values the others blend in
  const float* rope = nullptr;
  // delta rule / gated linear attention
  int taps = 1, rank = 0, low_rank_cfg = 0;                 // rank: inner size of the decay projection (from the tensors)
  float tau = 1.f;
  // feed-forward
  int ff = 0, experts = 0, top = 0, tile_rows = 32;
  float limit = 0.f;
  // weights: projections in the operand type (bf16 | f32), vectors f32
  float *norm1 = nullptr, *norm2 = nullptr, *qn = nullptr, *kn = nullptr, *sink = nullptr, *lambda = nullptr, *router_b = nullptr;
  float *conv_w = nullptr, *a_log = nullptr, *dt_bias = nullptr, *o_norm = nullptr, *a2T = nullptr, *a2_b = nullptr;
  void *in = nullptr, *o = nullptr, *a1 = nullptr;          // packed input projection (a1: first decay step until it is packed behind it)
  void *gu = nullptr, *down = nullptr;                      // dense: [gate rows | up rows], down
  void *router = nullptr, *egu = nullptr, *edown = nullptr; // experts: [E][gate rows | up rows][W], [E][W][ff]
  // columns of the packed input projection (f32 rows, padded to 8):
  //   attention [q | k | v | gate], delta [q | k | v | gate | beta | decay], gla [q | k | v | gate | a1]
  int k_heads() const { return mix == kGla ? H : G; }
  int q_cols() const { return (mix == kAttention ? H : k_heads()) * D; }
  int k_cols() const { return k_heads() * D; }
  int v_cols() const { return (mix == kAttention ? G : H) * V; }
  int g_cols() const { return mix == kAttention ? H : H * V; }
  int qkv() const { return q_cols() + k_cols() + v_cols(); }
  int base_cols() const { return qkv() + g_cols() + (mix == kDelta ? 2 * H : 0); }
  int in_cols() const { return base_cols() + (mix == kGla ? rank : 0); }
};

struct LayerState {
  void *kc = nullptr, *vc = nullptr;     // attention cache
  float *S = nullptr, *conv = nullptr;   // [slots, H, D, V], [slots, taps - 1, channels]
};

class Kalesun : public ModelBase {
 public:
  int vocab_ = 0, width_ = 0;
  float eps_ = 1e-5f, alpha_ = 1.f;
  std::vector<Layer> layers_;
  std::vector<LayerState> state_;
  std::set<std::string> optional_;       // tensors a checkpoint may carry although nothing reads them
  void* embed_ = nullptr;
  float* final_norm_ = nullptr;
  std::map<std::array<double, 6>, float*> rope_tables_;
  // activations
  float *h_ = nullptr, *proj_ = nullptr, *v_first_ = nullptr, *conv_out_ = nullptr, *decay_ = nullptr, *y_ = nullptr, *route_ = nullptr, *topk_w_ = nullptr;
  int32_t *topk_idx_ = nullptr, *row_token_ = nullptr, *tile_expert_ = nullptr, *slot_row_ = nullptr;
  void *x_ = nullptr, *q_ = nullptr, *mix_in_ = nullptr, *sub_out_ = nullptr, *gu_buf_ = nullptr, *act_ = nullptr, *xg_ = nullptr, *eout_ = nullptr,
       *head_in_ = nullptr;
  int head_rows_ = 0, max_rows_ = 0, vf_cols_ = 0;

  int vocab() const override { return vocab_; }
  int hidden() const override { return width_; }
  int layer_runs() const override { return static_cast<int>(layers_.size()); }
  bool recurrent_state() const override {
    for (const Layer& L : layers_) if (L.mix != kAttention) return true;
    return false;
  }

  int parse(const json::Value& c) {
    vocab_ = c["vocab"].need_int("vocab");
    width_ = c["width"].need_int("width");
    eps_ = static_cast<float>(c["norm"]["eps"].as_double(1e-5));
    alpha_ = static_cast<float>(c["postln_alpha"].need_double("postln_alpha"));
    const json::Value& ls = c["layers"];
    NVLLM_CHECK_ARG(ls.is_array() && ls.size() > 0 && vocab_ > 0 && width_ > 0, NVLLM_ERR_ARG, "Kalesun config: layers / vocab / width");
    int source = -1;
    for (size_t i = 0; i < ls.size(); ++i) {
      const json::Value& l = ls[i];
      Layer L;
      const std::string type = l["type"].as_string();
      const json::Value& m = l["mixer"];
      L.H = m["heads"].need_int("mixer.heads");
      L.G = m["kv_heads"].as_int(L.H);
      L.D = m["dim"].need_int("mixer.dim");
      L.V = m["vdim"].as_int(L.D);
      NVLLM_CHECK_ARG(L.H > 0 && L.G > 0 && L.H % L.G == 0 && L.D > 0 && L.V > 0, NVLLM_ERR_ARG, "Kalesun config: layer %zu heads %d / %d, dim %d, vdim %d",
                      i, L.H, L.G, L.D, L.V);
      if (type == "attention") {
        L.mix = kAttention;
        L.scale = static_cast<float>(m["scale"].need_double("mixer.scale"));
        L.window = m["mask"]["size"].as_int(0);
        L.keep_first = m["mask"]["keep_first"].as_int(0);
        L.rot_dims = m["rot"]["dims"].as_int(0);
        L.rot_base = m["rot"]["base"].as_double(10000.0);
        const json::Value& sc = m["rot"]["scaling"];
        if (!sc.is_null())
          L.rot_scaling = {sc["factor"].need_double("rot.scaling.factor"), sc["low"].need_double("rot.scaling.low"),
                           sc["high"].need_double("rot.scaling.high"), sc["original"].need_double("rot.scaling.original")};
        const auto& rs = L.rot_scaling;
        NVLLM_CHECK_ARG(L.V <= 512 && L.D <= 2048 && L.window >= 0 && L.keep_first >= 0, NVLLM_ERR_ARG,
                        "Kalesun config: layer %zu attention dim %d (<= 2048), vdim %d (<= 512), mask size %d, keep_first %d", i, L.D, L.V, L.window,
                        L.keep_first);
        NVLLM_CHECK_ARG(L.rot_dims >= 0 && L.rot_dims % 2 == 0 && L.rot_dims <= L.D && L.rot_base > 0, NVLLM_ERR_ARG,
                        "Kalesun config: layer %zu rot dims %d (even, <= dim %d)", i, L.rot_dims, L.D);
        NVLLM_CHECK_ARG(sc.is_null() || (rs[0] > 0 && rs[1] > 0 && rs[2] >= rs[1] && rs[3] > 0), NVLLM_ERR_ARG,
                        "Kalesun config: layer %zu rot scaling factor %g, low %g, high %g, original %g", i, rs[0], rs[1], rs[2], rs[3]);
        L.v_mix = m["v_mix"].as_int(0) != 0;
        if (L.v_mix && source < 0) {
          source = static_cast<int>(i);
          L.v_source = true;
        } else if (L.v_mix) {
          NVLLM_CHECK_ARG(layers_[source].G == L.G && layers_[source].V == L.V, NVLLM_ERR_ARG,
                          "Kalesun config: layer %zu mixes in the values of layer %d, which must have the same kv_heads and vdim", i, source);
        }
      } else if (type == "delta") {
        L.mix = kDelta;
        L.taps = m["conv"].need_int("mixer.conv");
        NVLLM_CHECK_ARG(L.D <= 512 && L.taps >= 1 && L.taps <= 16, NVLLM_ERR_ARG, "Kalesun config: layer %zu delta rule dim %d (<= 512), conv %d (1..16)",
                        i, L.D, L.taps);
      } else if (type == "gla") {
        L.mix = kGla;
        L.G = L.H;
        L.tau = static_cast<float>(m["tau"].need_double("mixer.tau"));
        L.low_rank_cfg = m["low_rank"].as_int(0);
        NVLLM_CHECK_ARG(L.D <= 512 && L.tau > 0, NVLLM_ERR_ARG, "Kalesun config: layer %zu gated linear attention dim %d (<= 512), tau %g", i, L.D,
                        static_cast<double>(L.tau));
      } else {
        NVLLM_CHECK_ARG(false, NVLLM_ERR_ARG, "Kalesun config: layer %zu has mixer type '%s' (known: attention, delta, gla)", i, type.c_str());
      }
      const json::Value& f = l["mlp"];
      if (!f.is_null()) {
        const std::string kind = f["kind"].as_string("dense");
        if (kind == "dense") {
          L.ffk = kDense;
          L.ff = f["ff"].need_int("mlp.ff");
          L.limit = static_cast<float>(f["limit"].need_double("mlp.limit"));
          NVLLM_CHECK_ARG(L.ff > 0 && L.limit > 0, NVLLM_ERR_ARG, "Kalesun config: layer %zu feed-forward size %d, limit %g", i, L.ff, static_cast<double>(L.limit));
        } else if (kind == "moe") {
          L.ffk = kExperts;
          L.ff = f["expert"]["ff"].need_int("mlp.expert.ff");
          L.limit = static_cast<float>(f["expert"]["limit"].need_double("mlp.expert.limit"));
          L.experts = f["router"]["experts"].need_int("mlp.router.experts");
          L.top = f["router"]["top"].need_int("mlp.router.top");
          NVLLM_CHECK_ARG(L.ff > 0 && L.limit > 0 && L.experts > 0 && L.experts <= 3072 && L.top > 0 && L.top <= L.experts, NVLLM_ERR_ARG,
                          "Kalesun config: layer %zu experts %d (<= 3072), top %d, expert size %d, limit %g", i, L.experts, L.top, L.ff,
                          static_cast<double>(L.limit));
        } else {
          NVLLM_CHECK_ARG(false, NVLLM_ERR_ARG, "Kalesun config: layer %zu feed-forward kind '%s' (known: dense, moe)", i, kind.c_str());
        }
      }
      layers_.push_back(L);
    }
    return 0;
  }

  // rotary table shared by the layers that agree on base, dims and scaling: [max_pos, dims / 2] of (cos, sin), angles in f64
  int rope_table(Layer& L, cudaStream_t stream) {
    const auto& s = L.rot_scaling;
    const std::array<double, 6> key{L.rot_base, static_cast<double>(L.rot_dims), s[0], s[1], s[2], s[3]};
    auto it = rope_tables_.find(key);
    if (it == rope_tables_.end()) {
      float* tab = nullptr;
      RUN(dalloc(&tab, static_cast<size_t>(lim_.max_positions) * L.rot_dims));
      RUN(nvllm_rope_table_scaled(tab, lim_.max_positions, L.rot_dims, L.rot_base, s[0], s[1], s[2], s[3], stream));
      it = rope_tables_.emplace(key, tab).first;
    }
    L.rope = it->second;
    return 0;
  }

  int create(const ModelLimits& lim, cudaStream_t stream) override {
    lim_ = lim;
    dt_ = lim.dtype;
    esz_ = dt_ == NVLLM_F32 ? 4 : 2;
    const size_t W = width_, T = lim.max_tokens, slots = lim.max_seqs;
    RUN(oalloc(&embed_, static_cast<size_t>(vocab_) * W)); needed_.insert("embed");
    RUN(valloc(&final_norm_, W, "final.norm"));
    size_t m_q = 8, m_mix = 8, m_ch = 1, m_dec = 1, m_hv = 1, m_gu = 0, m_ff = 0, m_eff = 0, m_exp = 0, m_top = 0;
    state_.resize(layers_.size());
    const size_t rows = static_cast<size_t>(lim.num_blocks) * lim.block_size;
    bool mixed = false;
    for (size_t i = 0; i < layers_.size(); ++i) {
      Layer& L = layers_[i];
      LayerState& st = state_[i];
      const std::string p = "l" + std::to_string(i) + ".", a = p + "mix.";
      const size_t HD = static_cast<size_t>(L.H) * L.D, HV = static_cast<size_t>(L.H) * L.V;
      RUN(valloc(&L.norm1, W, p + "norm1"));
      RUN(oalloc(&L.in, static_cast<size_t>(L.mix == kGla ? L.base_cols() : pad8(L.base_cols())) * W, true));
      RUN(oalloc(&L.o, W * HV));
      for (const char* t : {"q", "k", "v", "g", "o"}) needed_.insert(a + t);
      m_mix = std::max(m_mix, HV);
      if (L.mix == kAttention) {
        RUN(valloc(&L.qn, L.D, a + "q.norm")); RUN(valloc(&L.kn, L.D, a + "k.norm")); RUN(valloc(&L.sink, L.H, a + "sink"));
        if (L.rot_dims > 0) RUN(rope_table(L, stream));
        RUN(oalloc(&st.kc, rows * L.G * L.D, true)); RUN(oalloc(&st.vc, rows * L.G * L.V, true));
        m_q = std::max(m_q, HD);
        if (L.v_source) {
          vf_cols_ = (L.G * L.V + 3) / 4 * 4;
          optional_.insert(a + "vmix");
        } else if (L.v_mix) {
          RUN(valloc(&L.lambda, 1, a + "vmix"));
          mixed = true;
        }
      } else {
        RUN(valloc(&L.o_norm, L.V, a + "norm"));
        RUN(dalloc(&st.S, slots * HD * L.V, sizeof(float), true));
        m_hv = std::max(m_hv, HV);
        if (L.mix == kDelta) {
          RUN(dalloc(&L.conv_w, static_cast<size_t>(L.qkv()) * L.taps));
          for (const char* t : {"q.conv", "k.conv", "v.conv", "a", "b"}) needed_.insert(a + t);
          RUN(valloc(&L.a_log, L.H, a + "A_log")); RUN(valloc(&L.dt_bias, L.H, a + "dt_bias"));
          RUN(dalloc(&st.conv, slots * std::max(1, L.taps - 1) * L.qkv(), sizeof(float), true));
          m_ch = std::max<size_t>(m_ch, L.qkv());
        } else {
          needed_.insert(a + "a1"); needed_.insert(a + "a2");
          RUN(valloc(&L.a2_b, HD, a + "a2.b"));
          m_dec = std::max(m_dec, HD);
        }
      }
      if (L.ffk != kNone) RUN(valloc(&L.norm2, W, p + "norm2"));
      if (L.ffk == kDense) {
        RUN(oalloc(&L.gu, static_cast<size_t>(2) * L.ff * W)); RUN(oalloc(&L.down, W * L.ff));
        for (const char* t : {"gate", "up", "down"}) needed_.insert(p + "mlp." + t);
        m_ff = std::max<size_t>(m_ff, L.ff);
        if (!glu_in_gemm(L)) m_gu = std::max<size_t>(m_gu, 2 * L.ff);
      } else if (L.ffk == kExperts) {
        const size_t E = L.experts;
        RUN(oalloc(&L.router, static_cast<size_t>(pad8(L.experts)) * W, true)); needed_.insert(p + "mlp.router");
        RUN(valloc(&L.router_b, E, p + "mlp.router.b"));
        RUN(oalloc(&L.egu, E * 2 * L.ff * W)); RUN(oalloc(&L.edown, E * W * L.ff));
        for (int e = 0; e < L.experts; ++e)
          for (const char* t : {"gate", "up", "down"}) needed_.insert(p + "mlp.e" + std::to_string(e) + "." + t);
        if (dt_ == NVLLM_BF16 && W % 64 == 0 && L.ff % 64 == 0) L.tile_rows = 128;  // experts on the tensor-core grouped GEMM
        max_rows_ = std::max(max_rows_, nvllm_moe_max_rows(lim.max_tokens, L.top, L.experts, L.tile_rows));
        m_eff = std::max<size_t>(m_eff, L.ff); m_exp = std::max<size_t>(m_exp, pad8(L.experts)); m_top = std::max<size_t>(m_top, L.top);
      }
    }
    RUN(dalloc(&h_, T * W)); RUN(oalloc(&x_, T * W)); RUN(oalloc(&sub_out_, T * W)); RUN(oalloc(&q_, T * m_q)); RUN(oalloc(&mix_in_, T * m_mix));
    RUN(dalloc(&conv_out_, T * m_ch)); RUN(dalloc(&decay_, T * m_dec)); RUN(dalloc(&y_, T * m_hv));
    if (mixed) RUN(dalloc(&v_first_, T * vf_cols_));
    if (m_gu > 0) RUN(oalloc(&gu_buf_, T * m_gu));
    const size_t R = max_rows_;
    if (std::max(m_ff, m_eff) > 0) RUN(oalloc(&act_, std::max(T * m_ff, R * m_eff)));
    if (m_eff > 0) {
      RUN(dalloc(&route_, T * m_exp)); RUN(dalloc(&topk_idx_, T * m_top)); RUN(dalloc(&topk_w_, T * m_top));
      RUN(dalloc(&row_token_, R)); RUN(dalloc(&tile_expert_, R / 32 + 1)); RUN(dalloc(&slot_row_, T * m_top));
      RUN(oalloc(&xg_, R * W)); RUN(oalloc(&eout_, R * W));
    }
    NVLLM_CUDA(cudaStreamSynchronize(stream));
    return 0;
  }

  // dense feed-forward whose gate is applied in the GEMM's epilogue
  bool glu_in_gemm(const Layer& L) const { return dt_ == NVLLM_BF16 && L.ff % 128 == 0 && width_ % 64 == 0; }

  // ---- weights ---------------------------------------------------------------------------------------------------
  // The tensor's shape and where it goes.  kMat: operand matrix at (dst, element offset); kVec: f32 vector; kConv: taps, into the
  // packed [channels, taps] table at row `off`; kDown1 / kDown2: the two steps of a gla layer's decay projection, whose inner
  // size the tensors themselves decide (rows < 0 / cols < 0).
  enum Kind { kUnknown, kMat, kVec, kConv, kDown1, kDown2 };
  struct Target { Kind kind = kUnknown; void* dst = nullptr; size_t off = 0; int64_t rows = 0, cols = 0; int layer = -1; };
  Target target_of(const std::string& name) const {
    const int64_t W = width_;
    Target t;
    auto mat = [&](void* d, size_t off, int64_t r, int64_t c) { t.kind = kMat; t.dst = d; t.off = off; t.rows = r; t.cols = c; return t; };
    auto vec = [&](float* d, int64_t n) { t.kind = kVec; t.dst = d; t.rows = 1; t.cols = n; return t; };
    auto conv = [&](float* d, int64_t ch0, int64_t ch, int taps) { t.kind = kConv; t.dst = d; t.off = ch0; t.rows = ch; t.cols = taps; return t; };
    if (name == "embed") return mat(embed_, 0, vocab_, W);
    if (name == "final.norm") return vec(final_norm_, W);
    if (name.size() < 4 || name[0] != 'l') return t;
    const size_t dot = name.find('.');
    if (dot == std::string::npos) return t;
    const int li = atoi(name.substr(1, dot - 1).c_str());
    if (li < 0 || li >= static_cast<int>(layers_.size())) return t;
    const Layer& L = layers_[li];
    t.layer = li;
    const std::string rest = name.substr(dot + 1);
    const int64_t HV = static_cast<int64_t>(L.H) * L.V, q = L.q_cols(), k = L.k_cols(), qkv = L.qkv();
    if (rest == "norm1") return vec(L.norm1, W);
    if (rest == "norm2") return vec(L.norm2, W);
    if (rest == "mix.q") return mat(L.in, 0, q, W);
    if (rest == "mix.k") return mat(L.in, q * W, k, W);
    if (rest == "mix.v") return mat(L.in, (q + k) * W, L.v_cols(), W);
    if (rest == "mix.g") return mat(L.in, qkv * W, L.g_cols(), W);
    if (rest == "mix.o") return mat(L.o, 0, W, HV);
    if (L.mix == kAttention) {
      if (rest == "mix.q.norm") return vec(L.qn, L.D);
      if (rest == "mix.k.norm") return vec(L.kn, L.D);
      if (rest == "mix.sink") return vec(L.sink, L.H);
      if (rest == "mix.vmix") return vec(L.lambda, 1);
    } else if (rest == "mix.norm") {
      return vec(L.o_norm, L.V);
    }
    if (L.mix == kDelta) {
      if (rest == "mix.q.conv") return conv(L.conv_w, 0, q, L.taps);
      if (rest == "mix.k.conv") return conv(L.conv_w, q, k, L.taps);
      if (rest == "mix.v.conv") return conv(L.conv_w, q + k, HV, L.taps);
      if (rest == "mix.b") return mat(L.in, (qkv + HV) * W, L.H, W);
      if (rest == "mix.a") return mat(L.in, (qkv + HV + L.H) * W, L.H, W);
      if (rest == "mix.A_log") return vec(L.a_log, L.H);
      if (rest == "mix.dt_bias") return vec(L.dt_bias, L.H);
    } else if (L.mix == kGla) {
      if (rest == "mix.a1") { t.kind = kDown1; t.rows = -1; t.cols = W; return t; }
      if (rest == "mix.a2") { t.kind = kDown2; t.rows = static_cast<int64_t>(L.H) * L.D; t.cols = -1; return t; }
      if (rest == "mix.a2.b") return vec(L.a2_b, static_cast<int64_t>(L.H) * L.D);
    }
    if (L.ffk == kDense) {
      if (rest == "mlp.gate") return mat(L.gu, 0, L.ff, W);
      if (rest == "mlp.up") return mat(L.gu, static_cast<size_t>(L.ff) * W, L.ff, W);
      if (rest == "mlp.down") return mat(L.down, 0, W, L.ff);
    } else if (L.ffk == kExperts) {
      if (rest == "mlp.router") return mat(L.router, 0, L.experts, W);
      if (rest == "mlp.router.b") return vec(L.router_b, L.experts);
      if (rest.compare(0, 5, "mlp.e") == 0) {
        const size_t d2 = rest.find('.', 5);
        if (d2 == std::string::npos) return t;
        const int e = atoi(rest.substr(5, d2 - 5).c_str());
        if (e < 0 || e >= L.experts || rest.substr(5, d2 - 5) != std::to_string(e)) return t;
        const std::string part = rest.substr(d2 + 1);
        const size_t gu = static_cast<size_t>(e) * 2 * L.ff * W;
        if (part == "gate") return mat(L.egu, gu, L.ff, W);
        if (part == "up") return mat(L.egu, gu + static_cast<size_t>(L.ff) * W, L.ff, W);
        if (part == "down") return mat(L.edown, static_cast<size_t>(e) * W * L.ff, W, L.ff);
      }
    }
    return t;
  }

  // Operand matrices and f32 vectors arrive as bf16 bit patterns.
  int load_weight(const char* name_c, const void* src_v, int64_t rows, int64_t cols, cudaStream_t st) override {
    NVLLM_CHECK_ARG(name_c && src_v, NVLLM_ERR_ARG, "load_weight: NULL");
    const std::string name(name_c);
    if (optional_.count(name)) return 0;
    NVLLM_CHECK_ARG(needed_.count(name), NVLLM_ERR_ARG, "load_weight: tensor '%s' is not part of this model", name_c);
    Target t = target_of(name);
    NVLLM_CHECK_ARG(t.kind != kUnknown, NVLLM_ERR_ARG, "load_weight: unknown tensor '%s'", name_c);
    const uint16_t* src = static_cast<const uint16_t*>(src_v);
    if (t.kind == kDown1 || t.kind == kDown2) {
      Layer& L = layers_[t.layer];
      const int64_t inner = t.kind == kDown1 ? rows : cols;
      NVLLM_CHECK_ARG(inner > 0 && (t.kind == kDown1 ? cols == t.cols : rows == t.rows), NVLLM_ERR_ARG, "load_weight(%s): got [%lld, %lld]", name_c,
                      (long long)rows, (long long)cols);
      NVLLM_CHECK_ARG(L.rank == 0 || L.rank == inner, NVLLM_ERR_ARG, "load_weight(%s): inner size %lld, the other step has %d", name_c, (long long)inner,
                      L.rank);
      L.rank = static_cast<int>(inner);
      if (t.kind == kDown1 && ready_) {
        RUN(put(L.in, static_cast<size_t>(L.base_cols()) * width_, src, static_cast<size_t>(rows) * cols, st));
      } else if (t.kind == kDown1) {
        if (L.a1 == nullptr) RUN(oalloc(&L.a1, static_cast<size_t>(rows) * cols));
        RUN(put(L.a1, 0, src, static_cast<size_t>(rows) * cols, st));
      } else {
        if (L.a2T == nullptr) RUN(dalloc(&L.a2T, static_cast<size_t>(rows) * cols));
        RUN(putf(L.a2T, src, rows, cols, true, st));
      }
    } else {
      NVLLM_CHECK_ARG(rows * cols == t.rows * t.cols && (t.kind == kVec || (rows == t.rows && cols == t.cols)), NVLLM_ERR_ARG,
                      "load_weight(%s): expected [%lld, %lld], got [%lld, %lld]", name_c, (long long)t.rows, (long long)t.cols, (long long)rows,
                      (long long)cols);
      if (t.kind == kMat) RUN(put(t.dst, t.off, src, static_cast<size_t>(rows) * cols, st));
      else RUN(putf(static_cast<float*>(t.dst) + (t.kind == kConv ? t.off * cols : 0), src, rows, cols, false, st));
    }
    loaded_.insert(name);
    if (loaded_.size() == needed_.size() && !ready_) RUN(finish_load(st));
    return 0;
  }

  // Once every tensor is there: the gla layers' first decay step joins their input projection, so that one product serves
  // both, and the buffer that holds the projections' output gets its size.
  int finish_load(cudaStream_t st) {
    size_t m_proj = 8;
    for (Layer& L : layers_) {
      const size_t W = width_, n = pad8(L.in_cols());
      m_proj = std::max(m_proj, n);
      if (L.mix != kGla) continue;
      void* packed = nullptr;
      RUN(oalloc(&packed, n * W, true));
      const size_t base = static_cast<size_t>(L.base_cols()) * W;
      NVLLM_CUDA(cudaMemcpyAsync(packed, L.in, base * esz_, cudaMemcpyDeviceToDevice, st));
      NVLLM_CUDA(cudaMemcpyAsync(at(packed, base), L.a1, static_cast<size_t>(L.rank) * W * esz_, cudaMemcpyDeviceToDevice, st));
      NVLLM_CUDA(cudaStreamSynchronize(st));
      release(L.in); release(L.a1);
      L.in = packed; L.a1 = nullptr;
    }
    RUN(dalloc(&proj_, static_cast<size_t>(lim_.max_tokens) * m_proj));
    ready_ = true;
    return 0;
  }

  // Seeded synthetic weights (benchmarks, smoke runs): every needed tensor drawn on the host and sent through load_weight, so
  // that synthetic and checkpoint weights take the same path.
  int init_weights(uint64_t seed, float std, cudaStream_t st) override {
    std::vector<uint16_t> buf;
    uint64_t tid = 0;
    for (const std::string& name : needed_) {
      ++tid;
      Target t = target_of(name);
      NVLLM_CHECK_ARG(t.kind != kUnknown, NVLLM_ERR_STATE, "init_weights: no target for '%s'", name.c_str());
      if (t.kind == kDown1 || t.kind == kDown2) {   // inner size: the configuration's `low_rank`, else an eighth of the width
        const int r = layers_[t.layer].low_rank_cfg > 0 ? layers_[t.layer].low_rank_cfg : std::max(8, pad8(width_ / 8));
        if (t.rows < 0) t.rows = r;
        if (t.cols < 0) t.cols = r;
      }
      buf.resize(static_cast<size_t>(t.rows) * t.cols);
      const bool norm_w = name.find("norm") != std::string::npos, unit = ends(name, ".sink") || ends(name, ".router.b") || name == "embed" || t.kind == kConv;
      const bool shifted = ends(name, ".A_log") || ends(name, ".dt_bias"), lam = ends(name, ".vmix");
      for (size_t i = 0; i < buf.size(); ++i) {
        const float g = gauss(seed, tid, i);
        const float v = norm_w ? 1.0f + 0.1f * g : unit ? 0.5f * g : shifted ? -1.0f + 0.5f * g : lam ? 0.5f + 0.1f * g : g * std;
        buf[i] = f32_to_bf16_bits(v);
      }
      RUN(load_weight(name.c_str(), buf.data(), t.rows, t.cols, st));
    }
    return 0;
  }

  // ---- forward ---------------------------------------------------------------------------------------------------
  int forward(const StepView& v) override {
    void* st = v.stream;
    const int N = v.n_tokens, W = width_, S = v.n_seqs;
    launches = 0;
    NVLLM_CHECK_ARG(ready_, NVLLM_ERR_STATE, "Kalesun forward: weights are not loaded");
    NVLLM_CHECK_ARG(v.cu_tokens && v.tables && (v.seq_slots || !recurrent_state()), NVLLM_ERR_ARG,
                    "Kalesun forward: the step carries no token ranges / block tables / state slots");
    auto mk = [&](const char* name) { ++launches; if (v.mark) v.mark(v.mark_ctx, name); };
    auto lin = [&](void* y, const void* x, const void* w, int n, int k, int64_t ldy, int out_dt, const char* name) {
      const int rc = nvllm_linear(y, x, w, N, n, k, k, k, ldy, 1, 0, 0, 0, dt_, out_dt, st);
      mk(name);
      return rc;
    };
    // h = rms(alpha h + y) w, and what reads the stream next: the stream itself or, at the very end, the model's last norm of it
    auto join = [&](const float* w, const float* last) {
      const int rc = nvllm_rms_sum_norm(x_, h_, sub_out_, dt_, alpha_, w, last, N, W, eps_, dt_, st);
      mk(last ? "rms_sum_norm (+ final norm)" : "rms_sum_norm");
      return rc;
    };
    RUN(nvllm_embedding_stream(h_, x_, dt_, embed_, v.ids, N, W, vocab_, 1.0f, dt_, st)); mk("embedding_stream");
    for (size_t i = 0; i < layers_.size(); ++i) {
      const Layer& L = layers_[i];
      const LayerState& ls = state_[i];
      const bool last_layer = i + 1 == layers_.size();
      const int HD = L.H * L.D, HV = L.H * L.V, ld = pad8(L.in_cols()), qc = L.q_cols(), kc = L.k_cols(), qkv = L.qkv();
      if (L.mix == kAttention) {
        // [q | k | v | g]; head norms, rotation, value mixing and the cache store; attention in the window and over the kept
        // first keys, with the sink and the head gate
        const int GD = L.G * L.D, GV = L.G * L.V;
        RUN(lin(proj_, x_, L.in, ld, W, ld, NVLLM_F32, "attention q k v g projection"));
        float* vf = L.v_mix ? v_first_ : nullptr;
        RUN(nvllm_attn_norm_rotary_store(q_, HD, ls.kc, ls.vc, GD, GV, proj_, ld, L.qn, L.kn, eps_, v.positions, L.rope, L.rot_dims, 1, lim_.max_positions, vf,
                                         vf_cols_, L.lambda, v.slots, N, L.H, L.G, L.D, L.V, dt_, st)); mk("attn_norm_rotary_store");
        RUN(nvllm_masked_attention(mix_in_, HV, q_, HD, proj_ + qkv, ld, 1, ls.kc, ls.vc, GD, GV, v.tok_seq, v.positions, v.tables, v.table_cap,
                                   lim_.block_size, N, L.H, L.G, L.D, L.V, L.scale, 0.f, 0.f, 1, L.window, L.keep_first, L.sink, 0, nullptr, nullptr, 0,
                                   nullptr, 0, v.cu_tokens, S, dt_, st)); mk("masked_attention");
      } else if (L.mix == kDelta) {
        // [q | k | v | g | b | a]; the convolution + SiLU over (q, k, v); unit vectors, beta, the head's decay; the recurrence;
        // gated per-head norm
        float *gate = proj_ + qkv, *beta = gate + HV, *dec = beta + L.H;
        RUN(lin(proj_, x_, L.in, ld, W, ld, NVLLM_F32, "delta q k v g b a projection"));
        RUN(nvllm_causal_conv(conv_out_, qkv, proj_, ld, L.conv_w, nullptr, ls.conv, v.tok_seq, v.seq_slots, v.cu_tokens, v.positions, N, S, qkv, L.taps, 1,
                              st)); launches += L.taps > 1 ? 1 : 0; mk("causal_conv");
        RUN(nvllm_head_delta_prepare(conv_out_, qkv, conv_out_ + qc, qkv, beta, ld, dec, ld, L.a_log, L.dt_bias, N, L.H, L.G, L.D,
                                     1.0f / sqrtf(static_cast<float>(L.D)), 1e-6f, st)); mk("head_delta_prepare");
        RUN(nvllm_head_delta_recurrence(y_, HV, conv_out_, qkv, conv_out_ + qc, qkv, conv_out_ + qc + kc, qkv, dec, ld, beta, ld, ls.S, v.seq_slots,
                                        v.cu_tokens, v.positions, S, L.H, L.G, L.D, L.V, st)); mk("head_delta_recurrence");
        RUN(nvllm_gated_group_norm_act(mix_in_, HV, y_, HV, gate, ld, L.o_norm, 1, N, HV, L.H, eps_, 0, 0, dt_, st)); mk("gated_group_norm");
      } else {
        // [q | k | v | g | a1]; the second decay step; the recurrence; gated per-head norm
        float *gate = proj_ + qkv, *a1 = gate + HV;
        RUN(lin(proj_, x_, L.in, ld, W, ld, NVLLM_F32, "gla q k v g a1 projection"));
        RUN(nvllm_low_rank_decay(decay_, HD, a1, ld, L.a2T, L.a2_b, N, L.rank, HD, L.tau, st)); mk("low_rank_decay");
        RUN(nvllm_channel_recurrence(y_, HV, proj_, ld, proj_ + qc, ld, proj_ + qc + kc, ld, decay_, HD, 1.0f / sqrtf(static_cast<float>(L.D)), ls.S,
                                     v.seq_slots, v.cu_tokens, v.positions, S, L.H, L.H, L.D, L.V, st)); mk("channel_recurrence");
        RUN(nvllm_gated_group_norm_act(mix_in_, HV, y_, HV, gate, ld, L.o_norm, 1, N, HV, L.H, eps_, 0, 0, dt_, st)); mk("gated_group_norm");
      }
      RUN(lin(sub_out_, mix_in_, L.o, W, HV, W, dt_, "mixer output projection"));
      RUN(join(L.norm1, (last_layer && L.ffk == kNone) ? final_norm_ : nullptr));
      if (L.ffk == kDense) {
        if (glu_in_gemm(L)) {   // [N, 2 ff] never reaches HBM
          RUN(nvllm_gemm_glu_bf16(act_, x_, L.gu, N, L.ff, W, W, W, L.ff, L.limit, nullptr, 0, st)); mk("gate / up projection + clamped gate");
        } else {
          RUN(lin(gu_buf_, x_, L.gu, 2 * L.ff, W, 2 * L.ff, dt_, "gate / up projection"));
          RUN(nvllm_glu_clamped(act_, gu_buf_, N, L.ff, L.limit, dt_, st)); mk("glu_clamped");
        }
        RUN(lin(sub_out_, act_, L.down, W, L.ff, W, dt_, "down projection"));
      } else if (L.ffk == kExperts) {
        const int E = L.experts, lde = pad8(E);
        RUN(lin(route_, x_, L.router, lde, W, lde, NVLLM_F32, "router projection"));
        RUN(nvllm_moe_route_logits(topk_idx_, topk_w_, route_, lde, L.router_b, N, E, L.top, st)); mk("moe_route_logits");
        const int rows = nvllm_moe_max_rows(N, L.top, E, L.tile_rows);
        RUN(nvllm_moe_sort(row_token_, tile_expert_, slot_row_, topk_idx_, N, L.top, E, rows, L.tile_rows, st)); mk("moe_sort");
        if (L.tile_rows == 128) {
          RUN(nvllm_gather_rows(xg_, x_, row_token_, rows, W, N, dt_, st)); mk("expert row gather");
          RUN(nvllm_gemm_glu_bf16_grouped(act_, xg_, L.egu, rows, L.ff, W, E, W, W, L.ff, tile_expert_, L.limit, st)); mk("expert gate / up + clamped gate grouped GEMM");
          RUN(nvllm_gemm_bf16_grouped(eout_, act_, L.edown, rows, W, L.ff, E, L.ff, L.ff, W, tile_expert_, st)); mk("expert down grouped GEMM");
        } else {
          RUN(nvllm_linear_grouped(act_, x_, L.egu, rows, L.ff, W, W, W, L.ff, static_cast<int64_t>(2) * L.ff * W, row_token_, tile_expert_, 1, L.limit,
                                   dt_, dt_, st)); mk("expert gate / up + clamped gate grouped tile kernel");
          RUN(nvllm_linear_grouped(eout_, act_, L.edown, rows, W, L.ff, L.ff, L.ff, W, static_cast<int64_t>(W) * L.ff, nullptr, tile_expert_, 0, 0.f,
                                   dt_, dt_, st)); mk("expert down grouped tile kernel");
        }
        RUN(nvllm_moe_combine(sub_out_, eout_, x_, nullptr, topk_idx_, topk_w_, slot_row_, N, W, L.top, E, dt_, st)); mk("moe_combine");
      }
      if (L.ffk != kNone) RUN(join(L.norm2, last_layer ? final_norm_ : nullptr));
      if (v.layer_tap != nullptr && !v.capturing)
        NVLLM_CUDA(cudaMemcpyAsync(v.layer_tap + i * static_cast<size_t>(N) * W, h_, static_cast<size_t>(N) * W * 4, cudaMemcpyDeviceToHost,
                                   static_cast<cudaStream_t>(st)));
    }
    if (v.n_logit_rows > 0) {
      if (v.n_logit_rows > head_rows_) {
        NVLLM_CHECK_ARG(!v.capturing, NVLLM_ERR_STATE, "forward: logit rows grew inside a graph capture");
        NVLLM_CUDA(cudaStreamSynchronize(static_cast<cudaStream_t>(st)));
        head_rows_ = std::max(v.n_logit_rows, lim_.max_seqs);
        if (head_in_ != nullptr) release(head_in_);
        RUN(oalloc(&head_in_, static_cast<size_t>(head_rows_) * W));
      }
      RUN(nvllm_gather_rows(head_in_, x_, v.logit_rows, v.n_logit_rows, W, N, dt_, st)); mk("gather_rows");
      RUN(nvllm_linear(v.logits, head_in_, embed_, v.n_logit_rows, vocab_, W, W, W, vocab_, 1, 0, 0, 0, dt_, NVLLM_F32, st));
      mk("head projection (tied embedding)");
    }
    return 0;
  }
};

}  // namespace

ModelImpl* make_kalesun(const json::Value& cfg) {
  Kalesun* m = new Kalesun();
  if (m->parse(cfg) != 0) { delete m; return nullptr; }
  return m;
}

}  // namespace nvllm
