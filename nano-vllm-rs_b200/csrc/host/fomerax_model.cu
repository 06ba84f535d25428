// fomerax_model.cu — the Fomerax architecture on the runner's model interface (model.hpp).
//
// Fomerax is a decoder-only model on an f32 residual stream with an RMS norm before AND after every sublayer, and a small
// input of the token's own behind every layer,
//     x <- x + rms(mixer(rms(x) w1)) w1b;   x <- x + rms(ff(rms(x) w2)) w2b        (a layer may have no feed-forward)
//     x <- x + rms(Wp (gelu(Wg x) * e)) ws,   e = the layer's part of the token's row of a side table
// (the last step reads the stream itself).  Plain embedding, a final RMS norm and a tied output head.  Two kinds of mixer, in any
// order:
//   "attention"         grouped-query softmax attention over the paged cache (capped_attn.cu) without rotation: a query temperature
//                       that grows with the position, a soft cap on the scores and, after it, a slope per head
//                       (2^(-8 (h + 1) / heads)) times the distance taken off; one sigmoid gate per output value.
//   "latent_attention"  queries through an RMS-normed latent; ONE cached row [RMS-normed latent | rotated key part] per token, keys
//                       and values of the heads linear maps of the latent, the key part shared by the heads; a sliding window;
//                       rotary on neighbouring pairs with YaRN frequencies; one sigmoid gate per output value.  Portions and single
//                       tokens fold the key map into the query (latent_attn.cu); whole prompts compute keys and values of the step
//                       and run as ordinary windowed attention whose keys come in two parts (capped_attn.cu).
// Feed-forward: dense with a gelu gate, or a mixture of SiLU-gated experts on sigmoid scores: the `top` largest are used, the score
// multiplies the expert's INPUT (applied to the products' f32 accumulators) and the outputs are added as they are.
//
// bf16 engines: weights, projections' operands, sublayer outputs, q and the cache in bf16 with f32 accumulation; the residual,
// norms, scores, softmax, rotary angles and router in f32.  f32 engines: everything in f32.
//
// config.json keys: vocab, width, norm.eps, token_side.dim (absent: no token input), layers[] of {type, mixer, mlp}.
// layers[i].mixer by type: attention: heads, kv_heads, dim, vdim, scale, softcap, q_temp.{coef,every};
// latent_attention: heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, mask.size, rot.{base,dims,scaling.{factor,fast,slow,original}}.
// layers[i].mlp: null | {kind "dense", ff} | {kind "moe", expert.ff, router.{experts,top}}.
// tensors: embed, side.embed, final.norm, l<i>.norm{1,1b,2,2b}, l<i>.mix.{q,k,v,g,o} (attention),
// l<i>.mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,g,o} (latent), l<i>.mlp.{gate,up,down} (dense), l<i>.mlp.router,
// l<i>.mlp.e<k>.{gate,up,down} (experts), l<i>.side.{gate,proj,norm}.
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

enum MixKind { kAttention = 0, kLatent = 1 };
enum FfKind { kNone = 0, kDense = 1, kExperts = 2 };

struct Layer {
  int mix = kAttention, ffk = kNone;
  int H = 0, G = 0, D = 0, V = 0;            // latent: D unrotated query / key values per head
  float scale = 1.f;
  // attention
  float softcap = 0.f, temp_coef = 0.f;
  int temp_every = 1;
  const float* slopes = nullptr;
  // latent attention
  int window = 0, q_rank = 0, kv_rank = 0, rot = 0, rot_dims = 0;
  double rot_base = 10000.0;
  std::array<double, 4> yarn{0.0, 1.0, 1.0, 1.0};   // factor (0: plain rotary), fast, slow, original
  const float* rope = nullptr;
  // feed-forward
  int ff = 0, experts = 0, top = 0, tile_rows = 32;
  // weights: projections in the operand type (bf16 | f32), vectors f32
  float *norm1 = nullptr, *norm1b = nullptr, *norm2 = nullptr, *norm2b = nullptr, *side_norm = nullptr, *dq_norm = nullptr, *dkv_norm = nullptr;
  void *in = nullptr, *o = nullptr;                          // packed input projection, output projection
  void *uq = nullptr, *ukT = nullptr, *uv = nullptr;         // ukT: per head [kv_rank, D]
  void* ukv = nullptr;                                       // [uk | uv] as stored: keys and values of whole prompts
  void *gu = nullptr, *down = nullptr;                       // dense: [gate rows | up rows], down
  void *router = nullptr, *egu = nullptr, *edown = nullptr;  // experts: [E][gate rows | up rows][W], [E][W][ff]
  void *side_gate = nullptr, *side_proj = nullptr;
  // columns of the packed input projection (f32 rows, padded to 8): attention [q | k | v | gate], latent [dq | latent | key part | gate]
  int q_head() const { return D + rot; }
  int g_off() const { return mix == kAttention ? H * D + G * D + G * V : q_rank + kv_rank + rot; }
  int in_cols() const { return g_off() + H * V; }
  int cache_row() const { return pad8(kv_rank + rot); }
};

struct LayerCache { void *kc = nullptr, *vc = nullptr, *lat = nullptr; };

class Fomerax : public ModelBase {
 public:
  int vocab_ = 0, width_ = 0, side_ = 0;
  float eps_ = 1e-5f;
  std::vector<Layer> layers_;
  std::vector<LayerCache> cache_;
  void *embed_ = nullptr, *side_embed_ = nullptr;
  float* final_norm_ = nullptr;
  std::map<std::array<double, 6>, float*> rope_tables_;
  std::map<int, float*> slope_tables_;
  // activations
  float *h_ = nullptr, *proj_ = nullptr, *q_abs_ = nullptr, *route_ = nullptr, *topk_w_ = nullptr, *row_w_ = nullptr, *side_pre_ = nullptr, *lat_ws_ = nullptr;
  size_t lat_ws_bytes_ = 0;
  int32_t *topk_idx_ = nullptr, *row_token_ = nullptr, *tile_expert_ = nullptr, *slot_row_ = nullptr;
  void *x_ = nullptr, *q_ = nullptr, *cq_ = nullptr, *c_dense_ = nullptr, *kv_ = nullptr, *o_lat_ = nullptr, *mix_in_ = nullptr, *sub_out_ = nullptr,
       *gu_buf_ = nullptr, *act_ = nullptr, *xg_ = nullptr, *eout_ = nullptr, *side_in_ = nullptr, *head_in_ = nullptr;
  int head_rows_ = 0, max_rows_ = 0;

  int vocab() const override { return vocab_; }
  int hidden() const override { return width_; }
  int layer_runs() const override { return static_cast<int>(layers_.size()); }

  int parse(const json::Value& c) {
    vocab_ = c["vocab"].need_int("vocab");
    width_ = c["width"].need_int("width");
    eps_ = static_cast<float>(c["norm"]["eps"].need_double("norm.eps"));
    if (!c["token_side"].is_null()) {
      side_ = c["token_side"]["dim"].need_int("token_side.dim");
      NVLLM_CHECK_ARG(side_ > 0, NVLLM_ERR_ARG, "Fomerax config: token_side.dim %d", side_);
    }
    const json::Value& ls = c["layers"];
    NVLLM_CHECK_ARG(ls.is_array() && ls.size() > 0 && vocab_ > 0 && width_ > 0, NVLLM_ERR_ARG, "Fomerax config: layers / vocab / width");
    for (size_t i = 0; i < ls.size(); ++i) {
      const json::Value& l = ls[i];
      Layer L;
      const std::string type = l["type"].as_string();
      const json::Value& m = l["mixer"];
      L.H = m["heads"].need_int("mixer.heads");
      L.D = m["dim"].need_int("mixer.dim");
      L.V = m["vdim"].as_int(L.D);
      L.scale = static_cast<float>(m["scale"].need_double("mixer.scale"));
      NVLLM_CHECK_ARG(L.H > 0 && L.D > 0 && L.V > 0, NVLLM_ERR_ARG, "Fomerax config: layer %zu heads %d, dim %d, vdim %d", i, L.H, L.D, L.V);
      if (type == "attention") {
        L.mix = kAttention;
        L.G = m["kv_heads"].as_int(L.H);
        L.softcap = static_cast<float>(m["softcap"].as_double(0.0));
        L.temp_coef = static_cast<float>(m["q_temp"]["coef"].as_double(0.0));
        L.temp_every = m["q_temp"]["every"].as_int(1);
        NVLLM_CHECK_ARG(L.G > 0 && L.H % L.G == 0 && L.V <= 512 && L.D <= 2048, NVLLM_ERR_ARG,
                        "Fomerax config: layer %zu attention heads %d / %d, dim %d (<= 2048), vdim %d (<= 512)", i, L.H, L.G, L.D, L.V);
        NVLLM_CHECK_ARG(L.softcap >= 0.f && L.temp_every > 0, NVLLM_ERR_ARG, "Fomerax config: layer %zu softcap %g, q_temp.every %d", i,
                        static_cast<double>(L.softcap), L.temp_every);
      } else if (type == "latent_attention") {
        L.mix = kLatent;
        L.G = 1;
        L.rot = m["rot_dim"].need_int("mixer.rot_dim");
        L.q_rank = m["q_rank"].need_int("mixer.q_rank");
        L.kv_rank = m["kv_rank"].need_int("mixer.kv_rank");
        L.window = m["mask"]["size"].as_int(0);
        L.rot_dims = m["rot"]["dims"].as_int(L.rot);
        L.rot_base = m["rot"]["base"].as_double(10000.0);
        NVLLM_CHECK_ARG(L.q_rank > 0 && L.kv_rank > 0 && L.kv_rank <= 1024 && L.window >= 0, NVLLM_ERR_ARG,
                        "Fomerax config: layer %zu latent attention q_rank %d, kv_rank %d (<= 1024), mask size %d", i, L.q_rank, L.kv_rank, L.window);
        NVLLM_CHECK_ARG(L.rot >= 0 && L.rot_dims >= 0 && L.rot_dims % 2 == 0 && L.rot_dims <= L.rot && L.rot_base > 0, NVLLM_ERR_ARG,
                        "Fomerax config: layer %zu rot dims %d (even, <= rot_dim %d)", i, L.rot_dims, L.rot);
        const json::Value& sc = m["rot"]["scaling"];
        if (!sc.is_null()) {
          L.yarn = {sc["factor"].need_double("rot.scaling.factor"), sc["fast"].need_double("rot.scaling.fast"), sc["slow"].need_double("rot.scaling.slow"),
                    sc["original"].need_double("rot.scaling.original")};
          NVLLM_CHECK_ARG(L.yarn[0] > 0 && L.yarn[1] > 0 && L.yarn[2] > 0 && L.yarn[3] > 0 && L.rot_base > 1.0, NVLLM_ERR_ARG,
                          "Fomerax config: layer %zu rot scaling factor %g, fast %g, slow %g, original %g, base %g (> 1)", i, L.yarn[0], L.yarn[1], L.yarn[2],
                          L.yarn[3], L.rot_base);
        }
      } else {
        NVLLM_CHECK_ARG(false, NVLLM_ERR_ARG, "Fomerax config: layer %zu has mixer type '%s' (known: attention, latent_attention)", i, type.c_str());
      }
      const json::Value& f = l["mlp"];
      if (!f.is_null()) {
        const std::string kind = f["kind"].as_string("dense");
        if (kind == "dense") {
          L.ffk = kDense;
          L.ff = f["ff"].need_int("mlp.ff");
          NVLLM_CHECK_ARG(L.ff > 0, NVLLM_ERR_ARG, "Fomerax config: layer %zu feed-forward size %d", i, L.ff);
        } else if (kind == "moe") {
          L.ffk = kExperts;
          L.ff = f["expert"]["ff"].need_int("mlp.expert.ff");
          L.experts = f["router"]["experts"].need_int("mlp.router.experts");
          L.top = f["router"]["top"].need_int("mlp.router.top");
          NVLLM_CHECK_ARG(L.ff > 0 && L.experts > 0 && L.experts <= 3072 && L.top > 0 && L.top <= L.experts, NVLLM_ERR_ARG,
                          "Fomerax config: layer %zu experts %d (<= 3072), top %d, expert size %d", i, L.experts, L.top, L.ff);
        } else {
          NVLLM_CHECK_ARG(false, NVLLM_ERR_ARG, "Fomerax config: layer %zu feed-forward kind '%s' (known: dense, moe)", i, kind.c_str());
        }
      }
      layers_.push_back(L);
    }
    return 0;
  }

  // rotary table shared by the layers that agree on base, dims and scaling: [max_pos, dims / 2] of (cos, sin), angles in f64
  int rope_table(Layer& L, cudaStream_t stream) {
    const auto& s = L.yarn;
    const std::array<double, 6> key{L.rot_base, static_cast<double>(L.rot_dims), s[0], s[1], s[2], s[3]};
    auto it = rope_tables_.find(key);
    if (it == rope_tables_.end()) {
      float* tab = nullptr;
      RUN(dalloc(&tab, static_cast<size_t>(lim_.max_positions) * L.rot_dims));
      if (s[0] > 0.0) RUN(nvllm_rope_table_yarn(tab, lim_.max_positions, L.rot_dims, L.rot_base, s[0], s[1], s[2], s[3], stream));
      else RUN(nvllm_rope_table_interleaved(tab, lim_.max_positions, L.rot_dims, L.rot_base, stream));
      it = rope_tables_.emplace(key, tab).first;
    }
    L.rope = it->second;
    return 0;
  }

  // slopes of the distance bias, one table per number of heads
  int slope_table(Layer& L, cudaStream_t stream) {
    auto it = slope_tables_.find(L.H);
    if (it == slope_tables_.end()) {
      std::vector<float> s(L.H);
      for (int h = 0; h < L.H; ++h) s[h] = static_cast<float>(std::exp2(-8.0 * (h + 1) / L.H));
      float* tab = nullptr;
      RUN(dalloc(&tab, s.size()));
      NVLLM_CUDA(cudaMemcpyAsync(tab, s.data(), s.size() * 4, cudaMemcpyHostToDevice, stream));
      NVLLM_CUDA(cudaStreamSynchronize(stream));
      it = slope_tables_.emplace(L.H, tab).first;
    }
    L.slopes = it->second;
    return 0;
  }

  // Whole prompts of a latent layer as windowed attention over keys and values of the step (see forward): sizes the kernel takes.
  bool can_unfold(const Layer& L) const {
    return dt_ == NVLLM_BF16 && L.D % 8 == 0 && L.rot % 8 == 0 && L.V % 8 == 0 && L.q_head() <= 192 && L.V <= 128;
  }
  // dense feed-forward whose gate is applied in the GEMM's epilogue
  bool gate_in_gemm(const Layer& L) const { return dt_ == NVLLM_BF16 && L.ff % 128 == 0 && width_ % 64 == 0; }

  int create(const ModelLimits& lim, cudaStream_t stream) override {
    lim_ = lim;
    dt_ = lim.dtype;
    esz_ = dt_ == NVLLM_F32 ? 4 : 2;
    const size_t W = width_, T = lim.max_tokens;
    RUN(oalloc(&embed_, static_cast<size_t>(vocab_) * W)); needed_.insert("embed");
    RUN(valloc(&final_norm_, W, "final.norm"));
    if (side_ > 0) { RUN(oalloc(&side_embed_, static_cast<size_t>(vocab_) * side_ * layers_.size())); needed_.insert("side.embed"); }
    size_t m_proj = 8, m_q = 8, m_cq = 0, m_mix = 8, m_lat = 0, m_row = 0, m_kv = 0, m_ws = 0, m_gu = 0, m_ff = 0, m_eff = 0, m_exp = 0, m_top = 0;
    cache_.resize(layers_.size());
    const size_t rows = static_cast<size_t>(lim.num_blocks) * lim.block_size;
    for (size_t i = 0; i < layers_.size(); ++i) {
      Layer& L = layers_[i];
      LayerCache& kv = cache_[i];
      const std::string p = "l" + std::to_string(i) + ".", a = p + "mix.";
      const size_t HV = static_cast<size_t>(L.H) * L.V, HQ = static_cast<size_t>(L.H) * L.q_head();
      RUN(valloc(&L.norm1, W, p + "norm1")); RUN(valloc(&L.norm1b, W, p + "norm1b"));
      RUN(oalloc(&L.in, static_cast<size_t>(pad8(L.in_cols())) * W, true));
      RUN(oalloc(&L.o, W * HV));
      needed_.insert(a + "g"); needed_.insert(a + "o");
      m_proj = std::max<size_t>(m_proj, pad8(L.in_cols())); m_q = std::max(m_q, HQ); m_mix = std::max(m_mix, HV);
      if (L.mix == kAttention) {
        for (const char* t : {"q", "k", "v"}) needed_.insert(a + t);
        RUN(slope_table(L, stream));
        RUN(oalloc(&kv.kc, rows * L.G * L.D, true)); RUN(oalloc(&kv.vc, rows * L.G * L.V, true));
      } else {
        const size_t R = L.kv_rank, HD = static_cast<size_t>(L.H) * L.D;
        for (const char* t : {"dq", "uq", "dkv", "uk", "uv"}) needed_.insert(a + t);
        RUN(valloc(&L.dq_norm, L.q_rank, a + "dq.norm")); RUN(valloc(&L.dkv_norm, R, a + "dkv.norm"));
        RUN(oalloc(&L.uq, HQ * L.q_rank)); RUN(oalloc(&L.ukT, HD * R)); RUN(oalloc(&L.uv, HV * R));
        if (L.rot_dims > 0) RUN(rope_table(L, stream));
        RUN(oalloc(&kv.lat, rows * L.cache_row(), true));
        if (can_unfold(L)) {
          RUN(oalloc(&L.ukv, (HD + HV) * R));
          m_kv = std::max(m_kv, HD + HV); m_row = std::max<size_t>(m_row, L.cache_row());
        }
        m_cq = std::max<size_t>(m_cq, L.q_rank); m_lat = std::max(m_lat, L.H * R); m_ws = std::max(m_ws, L.H * (R + 2));
      }
      if (L.ffk != kNone) { RUN(valloc(&L.norm2, W, p + "norm2")); RUN(valloc(&L.norm2b, W, p + "norm2b")); }
      if (L.ffk == kDense) {
        RUN(oalloc(&L.gu, static_cast<size_t>(2) * L.ff * W)); RUN(oalloc(&L.down, W * L.ff));
        for (const char* t : {"gate", "up", "down"}) needed_.insert(p + "mlp." + t);
        m_ff = std::max<size_t>(m_ff, L.ff);
        if (!gate_in_gemm(L)) m_gu = std::max<size_t>(m_gu, 2 * L.ff);
      } else if (L.ffk == kExperts) {
        const size_t E = L.experts;
        RUN(oalloc(&L.router, static_cast<size_t>(pad8(L.experts)) * W, true)); needed_.insert(p + "mlp.router");
        RUN(oalloc(&L.egu, E * 2 * L.ff * W)); RUN(oalloc(&L.edown, E * W * L.ff));
        for (int e = 0; e < L.experts; ++e)
          for (const char* t : {"gate", "up", "down"}) needed_.insert(p + "mlp.e" + std::to_string(e) + "." + t);
        if (dt_ == NVLLM_BF16 && W % 64 == 0 && L.ff % 64 == 0) L.tile_rows = 128;  // experts on the tensor-core grouped GEMM
        max_rows_ = std::max(max_rows_, nvllm_moe_max_rows(lim.max_tokens, L.top, L.experts, L.tile_rows));
        m_eff = std::max<size_t>(m_eff, L.ff); m_exp = std::max<size_t>(m_exp, pad8(L.experts)); m_top = std::max<size_t>(m_top, L.top);
      }
      if (side_ > 0) {
        RUN(oalloc(&L.side_gate, static_cast<size_t>(pad8(side_)) * W, true)); RUN(oalloc(&L.side_proj, W * side_));
        RUN(valloc(&L.side_norm, W, p + "side.norm"));
        needed_.insert(p + "side.gate"); needed_.insert(p + "side.proj");
      }
    }
    RUN(dalloc(&h_, T * W)); RUN(oalloc(&x_, T * W)); RUN(oalloc(&sub_out_, T * W)); RUN(dalloc(&proj_, T * m_proj)); RUN(oalloc(&q_, T * m_q));
    RUN(oalloc(&mix_in_, T * m_mix));
    if (m_cq > 0) {
      RUN(oalloc(&cq_, T * m_cq)); RUN(dalloc(&q_abs_, T * m_lat)); RUN(oalloc(&o_lat_, T * m_lat));
      lat_ws_bytes_ = std::min<size_t>(T, 256) * 4 * m_ws * sizeof(float);   // partial softmaxes of single tokens: (tokens <= 256) x 4 splits
      RUN(dalloc(&lat_ws_, lat_ws_bytes_ / sizeof(float)));
    }
    if (m_kv > 0) { RUN(oalloc(&kv_, T * m_kv)); RUN(oalloc(&c_dense_, T * m_row, true)); }
    if (m_gu > 0) RUN(oalloc(&gu_buf_, T * m_gu));
    const size_t R = max_rows_;
    if (std::max(m_ff, m_eff) > 0) RUN(oalloc(&act_, std::max(T * m_ff, R * m_eff)));
    if (m_eff > 0) {
      RUN(dalloc(&route_, T * m_exp)); RUN(dalloc(&topk_idx_, T * m_top)); RUN(dalloc(&topk_w_, T * m_top)); RUN(dalloc(&row_w_, R));
      RUN(dalloc(&row_token_, R)); RUN(dalloc(&tile_expert_, R / 32 + 1)); RUN(dalloc(&slot_row_, T * m_top));
      RUN(oalloc(&xg_, R * W)); RUN(oalloc(&eout_, R * W));
    }
    if (side_ > 0) { RUN(dalloc(&side_pre_, T * pad8(side_))); RUN(oalloc(&side_in_, T * side_)); }
    NVLLM_CUDA(cudaStreamSynchronize(stream));
    return 0;
  }

  // ---- weights ---------------------------------------------------------------------------------------------------
  // The tensor's shape and where it goes.  kMat: operand matrix at (dst, element offset); kVec: f32 vector; kKeyMap / kValueMap: a
  // latent layer's key map (stored per head transposed) and value map, both also into the joint map of whole prompts.
  enum Kind { kUnknown, kMat, kVec, kKeyMap, kValueMap };
  struct Target { Kind kind = kUnknown; void* dst = nullptr; size_t off = 0; int64_t rows = 0, cols = 0; int layer = -1; };
  Target target_of(const std::string& name) const {
    const int64_t W = width_;
    Target t;
    auto mat = [&](void* d, size_t off, int64_t r, int64_t c, Kind k = kMat) { t.kind = k; t.dst = d; t.off = off; t.rows = r; t.cols = c; return t; };
    auto vec = [&](float* d, int64_t n) { t.kind = kVec; t.dst = d; t.rows = 1; t.cols = n; return t; };
    if (name == "embed") return mat(embed_, 0, vocab_, W);
    if (name == "side.embed") return mat(side_embed_, 0, vocab_, static_cast<int64_t>(side_) * layers_.size());
    if (name == "final.norm") return vec(final_norm_, W);
    if (name.size() < 4 || name[0] != 'l') return t;
    const size_t dot = name.find('.');
    if (dot == std::string::npos) return t;
    const int li = atoi(name.substr(1, dot - 1).c_str());
    if (li < 0 || li >= static_cast<int>(layers_.size())) return t;
    const Layer& L = layers_[li];
    t.layer = li;
    const std::string rest = name.substr(dot + 1);
    const int64_t HD = static_cast<int64_t>(L.H) * L.D, HV = static_cast<int64_t>(L.H) * L.V, GD = static_cast<int64_t>(L.G) * L.D,
                  GV = static_cast<int64_t>(L.G) * L.V, R = L.kv_rank;
    if (rest == "norm1") return vec(L.norm1, W);
    if (rest == "norm1b") return vec(L.norm1b, W);
    if (rest == "norm2") return vec(L.norm2, W);
    if (rest == "norm2b") return vec(L.norm2b, W);
    if (rest == "side.gate") return mat(L.side_gate, 0, side_, W);
    if (rest == "side.proj") return mat(L.side_proj, 0, W, side_);
    if (rest == "side.norm") return vec(L.side_norm, W);
    if (rest == "mix.g") return mat(L.in, static_cast<size_t>(L.g_off()) * W, HV, W);
    if (rest == "mix.o") return mat(L.o, 0, W, HV);
    if (L.mix == kAttention) {
      if (rest == "mix.q") return mat(L.in, 0, HD, W);
      if (rest == "mix.k") return mat(L.in, HD * W, GD, W);
      if (rest == "mix.v") return mat(L.in, (HD + GD) * W, GV, W);
    } else {
      if (rest == "mix.dq") return mat(L.in, 0, L.q_rank, W);
      if (rest == "mix.dkv") return mat(L.in, static_cast<size_t>(L.q_rank) * W, R + L.rot, W);
      if (rest == "mix.dq.norm") return vec(L.dq_norm, L.q_rank);
      if (rest == "mix.dkv.norm") return vec(L.dkv_norm, R);
      if (rest == "mix.uq") return mat(L.uq, 0, static_cast<int64_t>(L.H) * L.q_head(), L.q_rank);
      if (rest == "mix.uk") return mat(L.ukT, 0, HD, R, kKeyMap);
      if (rest == "mix.uv") return mat(L.uv, 0, HV, R, kValueMap);
    }
    if (L.ffk == kDense) {
      if (rest == "mlp.gate") return mat(L.gu, 0, L.ff, W);
      if (rest == "mlp.up") return mat(L.gu, static_cast<size_t>(L.ff) * W, L.ff, W);
      if (rest == "mlp.down") return mat(L.down, 0, W, L.ff);
    } else if (L.ffk == kExperts) {
      if (rest == "mlp.router") return mat(L.router, 0, L.experts, W);
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
    NVLLM_CHECK_ARG(needed_.count(name), NVLLM_ERR_ARG, "load_weight: tensor '%s' is not part of this model", name_c);
    const Target t = target_of(name);
    NVLLM_CHECK_ARG(t.kind != kUnknown, NVLLM_ERR_ARG, "load_weight: unknown tensor '%s'", name_c);
    NVLLM_CHECK_ARG(rows * cols == t.rows * t.cols && (t.kind == kVec || (rows == t.rows && cols == t.cols)), NVLLM_ERR_ARG,
                    "load_weight(%s): expected [%lld, %lld], got [%lld, %lld]", name_c, (long long)t.rows, (long long)t.cols, (long long)rows,
                    (long long)cols);
    const uint16_t* src = static_cast<const uint16_t*>(src_v);
    const size_t n = static_cast<size_t>(rows) * cols;
    if (t.kind == kVec) {
      RUN(putf(static_cast<float*>(t.dst), src, rows, cols, false, st));
    } else if (t.kind == kKeyMap) {   // [H * D, R] -> per head [R, D]: a query is folded through it, q_abs_h = Uk_h^T q_h
      const Layer& L = layers_[t.layer];
      std::vector<uint16_t> tr(n);
      for (int h = 0; h < L.H; ++h)
        for (int d = 0; d < L.D; ++d)
          for (int r = 0; r < L.kv_rank; ++r)
            tr[(static_cast<size_t>(h) * L.kv_rank + r) * L.D + d] = src[(static_cast<size_t>(h) * L.D + d) * L.kv_rank + r];
      RUN(put(t.dst, 0, tr.data(), n, st));
      if (L.ukv != nullptr) RUN(put(L.ukv, 0, src, n, st));
    } else {
      RUN(put(t.dst, t.off, src, n, st));
      if (t.kind == kValueMap && layers_[t.layer].ukv != nullptr)   // the value map also sits below the key map
        RUN(put(layers_[t.layer].ukv, static_cast<size_t>(layers_[t.layer].H) * layers_[t.layer].D * cols, src, n, st));
    }
    loaded_.insert(name);
    if (loaded_.size() == needed_.size()) ready_ = true;
    return 0;
  }

  // Seeded synthetic weights (benchmarks, smoke runs): every needed tensor drawn on the host and sent through load_weight, so
  // that synthetic and checkpoint weights take the same path.
  int init_weights(uint64_t seed, float std, cudaStream_t st) override {
    std::vector<uint16_t> buf;
    uint64_t tid = 0;
    for (const std::string& name : needed_) {
      ++tid;
      const Target t = target_of(name);
      NVLLM_CHECK_ARG(t.kind != kUnknown, NVLLM_ERR_STATE, "init_weights: no target for '%s'", name.c_str());
      buf.resize(static_cast<size_t>(t.rows) * t.cols);
      const bool norm_w = name.find("norm") != std::string::npos, table = ends(name, "embed");
      for (size_t i = 0; i < buf.size(); ++i) {
        const float g = gauss(seed, tid, i);
        buf[i] = f32_to_bf16_bits(norm_w ? 1.0f + 0.1f * g : table ? 0.5f * g : g * std);
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
    NVLLM_CHECK_ARG(ready_, NVLLM_ERR_STATE, "Fomerax forward: weights are not loaded");
    NVLLM_CHECK_ARG(v.cu_tokens && v.tables, NVLLM_ERR_ARG, "Fomerax forward: the step carries no token ranges / block tables");
    auto mk = [&](const char* name) { ++launches; if (v.mark) v.mark(v.mark_ctx, name); };
    auto lin = [&](void* y, const void* x, const void* w, int n, int k, int64_t ldx, int64_t ldy, int out_dt, const char* name) {
      const int rc = nvllm_linear(y, x, w, N, n, k, ldx, k, ldy, 1, 0, 0, 0, dt_, out_dt, st);
      mk(name);
      return rc;
    };
    // h += rms(y) * post, then what reads the stream next: rms(h) * pre, or (pre == NULL) the stream itself
    auto join = [&](const void* y, const float* post, const float* pre) {
      const int rc = nvllm_rms_residual_norm(x_, h_, y, dt_, post, pre, N, W, eps_, dt_, st);
      mk("rms_residual_norm");
      return rc;
    };
    RUN(nvllm_embedding_stream(h_, x_, dt_, embed_, v.ids, N, W, vocab_, 1.0f, dt_, st)); mk("embedding_stream");
    RUN(join(nullptr, nullptr, layers_[0].norm1));
    for (size_t i = 0; i < layers_.size(); ++i) {
      const Layer& L = layers_[i];
      const LayerCache& kv = cache_[i];
      const float* next = i + 1 < layers_.size() ? layers_[i + 1].norm1 : final_norm_;
      const float* behind_ff = side_ > 0 ? nullptr : next;      // the token input reads the stream itself
      const int HV = L.H * L.V, ld = pad8(L.in_cols());
      const float* gate = proj_ + L.g_off();
      if (L.mix == kAttention) {
        // [q | k | v | g]; the cache store; attention with temperature, cap, slopes and the gate
        const int HD = L.H * L.D, GD = L.G * L.D, GV = L.G * L.V;
        RUN(lin(proj_, x_, L.in, ld, W, W, ld, NVLLM_F32, "attention q k v g projection"));
        RUN(nvllm_attn_bias_store(q_, HD, kv.kc, kv.vc, GD, GV, proj_, ld, nullptr, nullptr, nullptr, v.slots, N, HD, GD, GV, dt_, st)); mk("attn_store");
        RUN(nvllm_extended_attention(mix_in_, HV, q_, HD, gate, ld, 0, kv.kc, kv.vc, GD, GV, v.tok_seq, v.positions, v.tables, v.table_cap, lim_.block_size,
                                     N, L.H, L.G, L.D, L.V, L.scale, L.softcap, L.temp_coef, L.temp_every, 0, 0, nullptr, 0, nullptr, nullptr, 0, nullptr, 0,
                                     L.slopes, nullptr, 0, 0, v.cu_tokens, S, dt_, st)); mk("sloped_attention");
      } else {
        // [dq | latent, key part | g]; both latents normed, the key part rotated, cache rows written; queries up and rotated
        const int R = L.kv_rank, HQ = L.H * L.q_head(), HD = L.H * L.D, HR = L.H * R, row = L.cache_row();
        RUN(lin(proj_, x_, L.in, ld, W, W, ld, NVLLM_F32, "latent dq dkv g projection"));
        // Whole prompts (every sequence starts at position 0, so all keys are the step's own tokens): keys and values per head are
        // computed from the step's latents and the layer runs as ordinary windowed attention over them, at a fraction of the
        // folded form's work (a key costs D + rot + V multiply-adds per head instead of 2 kv_rank + rot).
        const bool unfolded = v.whole_prompts && L.ukv != nullptr && knobs().latent_unfold && N >= 256;
        RUN(nvllm_latent_norm_store(cq_, L.q_rank, proj_, ld, L.q_rank, L.dq_norm, L.q_rank, R, L.rot, L.dkv_norm, eps_, v.positions, L.rope, L.rot_dims,
                                    lim_.max_positions, kv.lat, unfolded ? c_dense_ : nullptr, row, v.slots, N, dt_, st)); mk("latent_norm_store");
        RUN(lin(q_, cq_, L.uq, HQ, L.q_rank, L.q_rank, HQ, dt_, "query up-projection"));
        if (L.rot_dims > 0) {
          RUN(nvllm_rotate_tail(q_, HQ, v.positions, L.rope, L.rot_dims, lim_.max_positions, N, L.H, L.D, L.rot, dt_, st)); mk("rotate_tail (queries)");
        }
        // Per-head projections of the folded form: with many tokens every head is a tensor-core GEMM of its own; with few
        // (decoding) one batched launch of the mma.sync tile kernel beats `heads` launch latencies.
        const bool head_gemms = dt_ == NVLLM_BF16 && N >= 512 && L.D % 64 == 0 && R % 64 == 0 && L.V % 8 == 0 && L.rot % 8 == 0;
        if (unfolded) {
          const int kvn = HD + HV;
          RUN(lin(kv_, c_dense_, L.ukv, kvn, R, row, kvn, dt_, "key / value up-projection"));
          RUN(nvllm_extended_attention(mix_in_, HV, q_, HQ, gate, ld, 0, kv_, at(kv_, HD), kvn, kvn, v.tok_seq, v.positions, nullptr, v.table_cap,
                                       lim_.block_size, N, L.H, L.H, L.q_head(), L.V, L.scale, 0.f, 0.f, 1, L.window, 0, nullptr, 0, nullptr, nullptr, 0,
                                       nullptr, 0, nullptr, L.rot > 0 ? at(c_dense_, R) : nullptr, row, L.rot, v.cu_tokens, S, dt_, st));
          mk("window_attention (latent layer, whole prompts)");
        } else {
          if (head_gemms) {
            for (int hh = 0; hh < L.H; ++hh) {
              RUN(nvllm_gemm_bf16(q_abs_ + static_cast<size_t>(hh) * R, at(q_, static_cast<size_t>(hh) * L.q_head()),
                                  at(L.ukT, static_cast<size_t>(hh) * R * L.D), N, R, L.D, HQ, L.D, HR, NVLLM_F32, nullptr, 0, st));
              launches += hh > 0;
            }
            mk("q absorb (per-head GEMMs)");
          } else {
            RUN(nvllm_linear(q_abs_, q_, L.ukT, N, R, L.D, HQ, L.D, HR, L.H, L.q_head(), static_cast<int64_t>(R) * L.D, R, dt_, NVLLM_F32, st));
            mk("q absorb (per-head linear)");
          }
          RUN(nvllm_latent_window_attention(o_lat_, HR, q_abs_, HR, q_, HQ, v.tok_seq, v.positions, v.tables, v.table_cap, lim_.block_size, kv.lat, row, N,
                                            L.H, L.D, L.rot, R, L.scale, L.window, nullptr, nullptr, 0, lat_ws_, lat_ws_bytes_, dt_, st));
          mk("latent_window_attention");
          if (head_gemms) {
            for (int hh = 0; hh < L.H; ++hh) {
              RUN(nvllm_gemm_bf16(at(mix_in_, static_cast<size_t>(hh) * L.V), at(o_lat_, static_cast<size_t>(hh) * R),
                                  at(L.uv, static_cast<size_t>(hh) * L.V * R), N, L.V, R, HR, R, HV, NVLLM_BF16, nullptr, 0, st));
              launches += hh > 0;
            }
            mk("value up-projection (per-head GEMMs)");
            RUN(nvllm_sigmoid_gate(mix_in_, HV, gate, ld, N, HV, dt_, st)); mk("sigmoid_gate");
          } else {
            RUN(nvllm_linear_gated(mix_in_, o_lat_, L.uv, N, L.V, R, HR, R, HV, L.H, R, static_cast<int64_t>(L.V) * R, L.V, gate, ld, L.V, dt_, dt_, st));
            mk("value up-projection + gate (per-head linear)");
          }
        }
      }
      RUN(lin(sub_out_, mix_in_, L.o, W, HV, HV, W, dt_, "mixer output projection"));
      RUN(join(sub_out_, L.norm1b, L.ffk != kNone ? L.norm2 : behind_ff));
      if (L.ffk == kDense) {
        if (gate_in_gemm(L)) {   // [N, 2 ff] never reaches HBM
          RUN(nvllm_gemm_gated_bf16(act_, x_, L.gu, N, L.ff, W, W, W, L.ff, NVLLM_GATE_GELU, 0.f, nullptr, 0, st)); mk("gate / up projection + gelu gate");
        } else {
          RUN(lin(gu_buf_, x_, L.gu, 2 * L.ff, W, W, 2 * L.ff, dt_, "gate / up projection"));
          RUN(nvllm_ff_activation_params(act_, gu_buf_, N, L.ff, 3, nullptr, dt_, st)); mk("ff_activation (gelu gate)");
        }
        RUN(lin(sub_out_, act_, L.down, W, L.ff, L.ff, W, dt_, "down projection"));
      } else if (L.ffk == kExperts) {
        const int E = L.experts, lde = pad8(E);
        RUN(lin(route_, x_, L.router, lde, W, W, lde, NVLLM_F32, "router projection"));
        RUN(nvllm_moe_route_sigmoid(topk_idx_, topk_w_, route_, lde, nullptr, N, E, L.top, st)); mk("moe_route_sigmoid");
        const int rows = nvllm_moe_max_rows(N, L.top, E, L.tile_rows);
        RUN(nvllm_moe_sort_weighted(row_token_, row_w_, tile_expert_, slot_row_, topk_idx_, topk_w_, N, L.top, E, rows, L.tile_rows, st)); mk("moe_sort");
        if (L.tile_rows == 128) {
          RUN(nvllm_gather_rows(xg_, x_, row_token_, rows, W, N, dt_, st)); mk("expert row gather");
          RUN(nvllm_gemm_gated_bf16_grouped(act_, xg_, L.egu, rows, L.ff, W, E, W, W, L.ff, tile_expert_, NVLLM_GATE_SILU, 0.f, row_w_, st));
          mk("expert gate / up + silu gate grouped GEMM");
          RUN(nvllm_gemm_bf16_grouped(eout_, act_, L.edown, rows, W, L.ff, E, L.ff, L.ff, W, tile_expert_, st)); mk("expert down grouped GEMM");
        } else {
          RUN(nvllm_linear_grouped_scaled(act_, x_, L.egu, rows, L.ff, W, W, W, L.ff, static_cast<int64_t>(2) * L.ff * W, row_token_, row_w_, tile_expert_, 3,
                                          0.f, dt_, dt_, st)); mk("expert gate / up + silu gate grouped tile kernel");
          RUN(nvllm_linear_grouped(eout_, act_, L.edown, rows, W, L.ff, L.ff, L.ff, W, static_cast<int64_t>(W) * L.ff, nullptr, tile_expert_, 0, 0.f,
                                   dt_, dt_, st)); mk("expert down grouped tile kernel");
        }
        RUN(nvllm_moe_combine(sub_out_, eout_, x_, nullptr, topk_idx_, nullptr, slot_row_, N, W, L.top, E, dt_, st)); mk("moe_combine");
      }
      if (L.ffk != kNone) RUN(join(sub_out_, L.norm2b, behind_ff));
      if (side_ > 0) {
        // the token's own row of this layer, gated by the stream
        const int lds = pad8(side_);
        RUN(lin(side_pre_, x_, L.side_gate, lds, W, W, lds, NVLLM_F32, "token input gate projection"));
        RUN(nvllm_token_gate(side_in_, side_pre_, lds, side_embed_, static_cast<int64_t>(side_) * layers_.size(), static_cast<int64_t>(i) * side_, v.ids, vocab_,
                             N, side_, dt_, st)); mk("token_gate");
        RUN(lin(sub_out_, side_in_, L.side_proj, W, side_, side_, W, dt_, "token input projection"));
        RUN(join(sub_out_, L.side_norm, next));
      }
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

ModelImpl* make_fomerax(const json::Value& cfg) {
  Fomerax* m = new Fomerax();
  if (m->parse(cfg) != 0) { delete m; return nullptr; }
  return m;
}

}  // namespace nvllm
