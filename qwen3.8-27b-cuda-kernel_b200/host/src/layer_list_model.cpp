// Weights, cache, state and step of the layer-list architectures (see layer_list_model.h).
#include "layer_list_model.h"

#include <algorithm>

namespace qwen38 {

namespace {

constexpr int kMaxSplits = 64;
constexpr int kStatSplits = 8;
int up(int x, int to) { return int(align_up(x, to)); }

// The tensors of one design by name and expected shape; `at` reads one as fp32.
class TensorReader {
 public:
  explicit TensorReader(const ModelFile& f) : file_(f) {}
  void require(const std::string& name, std::vector<int64_t> shape) const {
    const TensorInfo& t = file_.tensor(name);
    QWEN38_CHECK(t.dtype == DType::BF16 || t.dtype == DType::F32, name, ": dtype ", dtype_name(t.dtype));
    auto text = [](const std::vector<int64_t>& s) {
      std::string o = "[";
      for (size_t i = 0; i < s.size(); ++i) o += (i ? ", " : "") + std::to_string(s[i]);
      return o + "]";
    };
    QWEN38_CHECK(t.shape == shape, name, ": shape ", text(t.shape), ", expected ", text(shape));
  }
  float at(const TensorInfo& t, int64_t i) const {
    const uint8_t* p = file_.data(t.offset, t.bytes).data();
    if (t.dtype == DType::F32) {
      float v;
      std::memcpy(&v, p + 4 * i, 4);
      return v;
    }
    uint16_t b;
    std::memcpy(&b, p + 2 * i, 2);
    return bf16_to_f32(b);
  }
  // `count` consecutive elements from element i as bf16
  void copy_bf16(const TensorInfo& t, int64_t i, int64_t count, q38_bf16* dst) const {
    const uint8_t* p = file_.data(t.offset, t.bytes).data();
    if (t.dtype == DType::BF16) std::memcpy(dst, p + 2 * i, size_t(2 * count));
    else
      for (int64_t k = 0; k < count; ++k) dst[k] = f32_to_bf16(at(t, i + k));
  }
  const ModelFile& file() const { return file_; }

 private:
  const ModelFile& file_;
};

struct Linear {
  std::vector<std::string> weights;             // stacked along the output
  std::vector<std::string> biases;              // one per weight, "" = none
  bool interleave = false;                      // two weights whose rows alternate
  // rows in heads (one size per weight): every head is padded with zero rows to a multiple of 16
  std::vector<int> heads_of = {};
};

struct LayerTensors {
  Linear in, out, up, down;
};

std::string mix(int i, const char* name) { return "l" + std::to_string(i) + ".mix." + name; }
std::string at_layer(int i, const char* name) { return "l" + std::to_string(i) + "." + name; }

LayerTensors names_of(const LayerSpec& l, int i, LayerListDesign::FeedForward ff) {
  LayerTensors t;
  auto w = [&](const char* n) { return mix(i, n); };
  switch (l.mixer) {
    case MixerKind::Attention:
      t.in = {{w("q"), w("k"), w("v")}, {w("q.b"), w("k.b"), w("v.b")}};
      t.out = {{w("o")}, {w("o.b")}};
      break;
    case MixerKind::MinGru:
      t.in = {{w("z"), w("x"), w("g")}, {w("z.b"), w("x.b"), ""}};
      t.out = {{w("o")}, {""}};
      break;
    case MixerKind::RgLru:
      t.in = {{w("y"), w("x")}, {w("y.b"), w("x.b")}};
      t.out = {{w("o")}, {""}};
      break;
    case MixerKind::Retention:
      t.in = {{w("q"), w("k"), w("v"), w("g")}, {"", "", "", ""}};
      t.out = {{w("o")}, {""}};
      break;
    case MixerKind::LatentAttention:
      t.in = {{w("dq"), w("dkv"), w("g")}, {"", "", ""}};
      t.out = {{w("o")}, {""}};
      break;
  }
  if (l.ff) {
    if (ff == LayerListDesign::FeedForward::Xielu) t.up = {{at_layer(i, "mlp.up")}, {""}};
    else t.up = {{at_layer(i, "mlp.gate"), at_layer(i, "mlp.up")}, {"", ""}, true};
    t.down = {{at_layer(i, "mlp.down")}, {""}};
  }
  return t;
}

struct StreamWeights {  // one sublayer's hyper-connection
  const float *in = nullptr, *out = nullptr, *mix = nullptr;
};

struct LayerWeightsDev {
  kernels::DenseWeight in{}, out{}, up{}, down{};
  float alpha_p = 0.0f, alpha_n = 0.0f;  // xIELU
  StreamWeights hc1, hc2;
  const float* decay_pow = nullptr;
  const float *q_gain = nullptr, *kv_gain = nullptr;
  kernels::DenseWeight uq{}, uk{}, uv{};  // latent attention; uk and uv hold one matrix per head
  kernels::DenseWeight ukv{};             // ... and all heads' keys, then values, from a latent (heads padded to 16)
  const float *norm1 = nullptr, *norm1b = nullptr, *norm2 = nullptr, *norm2b = nullptr;
  const float *v_mix = nullptr, *head_mix = nullptr;
  const double* inv_freq = nullptr;
  const float *conv_w = nullptr, *conv_b = nullptr, *gate_b = nullptr, *lam = nullptr;
  const q38_bf16* gate_w = nullptr;
  int block_ld = 0;
};

class LayerListModel final : public StepModel {
 public:
  LayerListModel(const ModelFile& f, const RunnerOptions& o, const LayerListDesign& d);

  size_t weight_bytes() const override { return weight_bytes_; }
  kernels::KvDtype resolve_kv_dtype(kernels::KvDtype d) const override {
    const kernels::KvDtype own = f32_ ? kernels::KvDtype::F32 : kernels::KvDtype::BF16;
    QWEN38_CHECK(d == kernels::KvDtype::Auto || d == own, cfg_.architecture, ": the KV cache has the activations' precision");
    return own;
  }
  size_t kv_page_bytes(kernels::KvDtype d) const override {
    size_t scores = 0;  // the decode kernels keep one page's scores of every head beside the pool
    if (score_heads_ > 0) scores = size_t(score_heads_) * kernels::kPageTokens * 4;
    return KvCache::page_bytes_all_layers(kv_layers_, d) + scores;
  }
  size_t state_bytes_per_slot() const override { return RecurrentStatePool::bytes_per_slot(rec_layers_, elem_); }
  void load_weights() override;
  std::unique_ptr<KvCache> make_kv(kernels::KvDtype d, int pages, int slots, int max_pages) const override {
    return std::make_unique<KvCache>(kv_layers_, d, pages, slots, max_pages);
  }
  void make_state(int slots) override { state_ = std::make_unique<RecurrentStatePool>(rec_layers_, elem_, slots); }
  void reset_slot(int slot, cudaStream_t s) override { state_->reset(slot, s); }
  void carve(Workspace& w, const StepContext& ctx) override;
  void prepare(const StepContext& ctx) override;
  void forward(const StepContext& ctx, const StepBatch& b) override;
  void head(const StepContext& ctx, const HeadRows& rows, float* logits) override;
  const kernels::GemmWorkspace* gemm_workspace() const override { return &gemm_ws_; }

 private:
  // weight upload; without an arena the sizes are only added up
  void visit_weights(DeviceArena* arena);
  template <typename T>
  const T* put(DeviceArena* arena, const std::vector<T>& v);
  kernels::DenseWeight put_linear(DeviceArena* arena, const Linear& l);
  kernels::DenseWeight put_heads(DeviceArena* arena, const std::string& name, int heads, int n_to, bool transpose);
  const float* put_f32(DeviceArena* arena, const std::string& name);
  const q38_bf16* put_bf16(DeviceArena* arena, const std::string& name);

  void gemm(const StepContext& ctx, const void* x, int ldx, int m, const kernels::DenseWeight& w, int kind, void* out, int ldo) {
    kernels::DenseEpilogue ep{};
    ep.kind = kind;
    ep.out = out;
    ep.ldo = ldo;
    kernels::dense_gemm(x, ldx, act_, m, w, ep, gemm_ws_, ctx.stream);
  }
  kernels::Norm norm(const float* gain) const {
    return {gain, design_.norm_gain_is_scalar ? 0 : 1, cfg_.rms_norm_eps, cfg_.norm_groups};
  }
  StreamWeights put_streams(DeviceArena* arena, int layer, const char* name);
  // A sublayer's output (y_) joins the residual, and the next sublayer's normed input is formed (unless there is none).
  struct Sublayer {
    const float* pre = nullptr;   // pre-norm gain, null = nothing follows
    const float* post = nullptr;  // post-norm gain
    StreamWeights hc;
  };
  Sublayer mixer_of(int run) const {
    const LayerWeightsDev& W = layers_[size_t(runs_[size_t(run)])];
    return {W.norm1, W.norm1b, W.hc1};
  }
  Sublayer feed_forward_of(int run) const {
    const LayerWeightsDev& W = layers_[size_t(runs_[size_t(run)])];
    return {W.norm2, W.norm2b, W.hc2};
  }
  void join_residual(const StepContext& ctx, int m, const Sublayer& done, const Sublayer& next);
  void feed_forward(const StepContext& ctx, int m, const LayerWeightsDev& W);
  void attention(const StepContext& ctx, const StepBatch& b, const LayerSpec& l, const LayerWeightsDev& W, int attn_i, bool first_values, bool blend);
  bool packs(const LatentAttentionSpec& a) const { return !f32_ && q38_packed_attention_fits(a.dim, a.vdim) != 0; }
  bool packing_pays(const LatentAttentionSpec& a, const StepBatch& b) const;
  void latent_attention(const StepContext& ctx, const StepBatch& b, const LayerSpec& l, const LayerWeightsDev& W, int attn_i);
  void recurrent(const StepContext& ctx, const StepBatch& b, const LayerSpec& l, const LayerWeightsDev& W, int rec_i);
  void retention(const StepContext& ctx, const StepBatch& b, const LayerSpec& l, const LayerWeightsDev& W,
                 const kernels::RecurrentStateDesc& st);

  TensorReader reader_;
  ModelConfig cfg_;
  LayerListDesign design_;
  bool f32_ = false;
  int act_ = Q38_ACT_BF16;
  size_t elem_ = 2;
  std::vector<int> runs_;  // layers in the order they run; a run's cache or state is the run's own
  int streams_ = 1;
  bool hyper_ = false;     // the weights have hyper-connections (otherwise one stream, plain sum)
  std::vector<KvLayerGeometry> kv_layers_;
  std::vector<RecurrentLayerGeometry> rec_layers_;
  int score_heads_ = 0;
  size_t weight_bytes_ = 0;

  DeviceArena arena_;
  std::vector<LayerWeightsDev> layers_;
  const q38_bf16 *embed_ = nullptr, *pos_ = nullptr;
  const float *final_norm_ = nullptr, *ones_ = nullptr;
  kernels::DenseWeight head_{};
  std::unique_ptr<RecurrentStatePool> state_;
  DeviceBuffer scores_;

  // activations; leading dimensions are multiples of 64 elements
  int ld_x_ = 0, ld_proj_ = 0, ld_mixer_ = 0, ld_ff_ = 0, max_q_ = 0, max_v_ = 0, max_heads_ = 0, max_rec_ = 0, max_attn_out_ = 0;
  float* residual_ = nullptr;
  uint8_t* x_ = nullptr;       // normed input of the sublayer
  uint8_t* proj_ = nullptr;    // the mixer's input projections
  uint8_t* mixer_ = nullptr;   // what enters the output projection
  uint8_t* ff_ = nullptr;
  float* y_ = nullptr;         // sublayer output before its post-norm
  uint8_t* q_ = nullptr;
  uint8_t* v_first_ = nullptr;
  float* stats_ = nullptr;
  float* partials_ = nullptr;
  float* rec_scratch_ = nullptr;
  uint8_t* qk_ = nullptr;      // retention: rotated queries and keys of a prefill step
  float* rec_o_ = nullptr;     // retention: outputs before their norm
  uint8_t* q_latent_ = nullptr;    // latent attention: normed query latents
  uint8_t* q_heads_ = nullptr;     // ... queries per head
  uint8_t* q_absorbed_ = nullptr;  // ... and in the space of the cached latents
  uint8_t* o_latent_ = nullptr;
  float* latent_partials_ = nullptr;
  uint8_t* packed_latents_ = nullptr;  // latents of a prefill step's contexts ...
  uint8_t* packed_kv_ = nullptr;       // ... and the heads' keys and values made from them
  int64_t packed_rows_ = 0;            // room for
  int ld_packed_ = 0, max_context_ = 0;
  size_t latent_partial_floats_ = 0;
  int ld_q_latent_ = 0, ld_q_heads_ = 0, max_absorbed_ = 0, max_latent_k_ = 0, max_rec_o_ = 0;
  size_t qk_bytes_per_token_ = 0;
  uint8_t* head_x_ = nullptr;
  kernels::GemmWorkspace gemm_ws_;
};

LayerListModel::LayerListModel(const ModelFile& f, const RunnerOptions& o, const LayerListDesign& d)
    : reader_(f), cfg_(f.config()), design_(d), f32_(o.compute == ComputeDtype::F32) {
  max_context_ = o.max_context;
  act_ = f32_ ? Q38_ACT_F32 : Q38_ACT_BF16;
  elem_ = f32_ ? 4 : 2;
  ld_x_ = up(cfg_.hidden_size, 64);
  runs_ = cfg_.layer_runs();
  hyper_ = cfg_.streams > 1 || (cfg_.streams == 1 && cfg_.num_layers > 0 && f.has_tensor(at_layer(0, "hc1.in")));
  streams_ = std::max(1, cfg_.streams);
  QWEN38_CHECK(!design_.post_norms || (streams_ == 1 && cfg_.norm_groups == 1 && cfg_.embedding_scale == 1.0f && cfg_.residual_mult == 1.0f),
               "post-norms go with one plain residual");
  int v_first = 0;
  for (const int run : runs_) {
    const LayerSpec& l = cfg_.layers[size_t(run)];
    if (l.mixer == MixerKind::Attention) {
      const AttentionSpec& a = l.attn;
      const KvLayerGeometry g{a.kv_heads, up(a.dim, 32), up(a.vdim, 8)};
      kv_layers_.push_back(g);
      if (!f32_) score_heads_ = std::max(score_heads_, a.heads);
      max_heads_ = std::max(max_heads_, a.heads);
      max_q_ = std::max(max_q_, a.heads * g.k_dim);
      max_attn_out_ = std::max(max_attn_out_, a.heads * g.v_dim);
      ld_proj_ = std::max(ld_proj_, up(a.heads * a.dim + a.kv_heads * (a.dim + a.vdim), 64));
      ld_mixer_ = std::max(ld_mixer_, up(a.heads * a.vdim, 64));
      if (a.value_mix) {
        QWEN38_CHECK(v_first == 0 || v_first == a.kv_heads * a.vdim, "layers that blend values need value heads of one total size");
        v_first = a.kv_heads * a.vdim;
      }
    } else if (l.mixer == MixerKind::LatentAttention) {
      const LatentAttentionSpec& a = l.latent;
      const KvLayerGeometry g{1, up(a.kv_rank, 32), 0};
      kv_layers_.push_back(g);
      ld_proj_ = std::max(ld_proj_, up(a.q_rank + a.kv_rank + a.heads * a.vdim, 64));
      ld_mixer_ = std::max(ld_mixer_, up(a.heads * a.vdim, 64));
      ld_q_latent_ = std::max(ld_q_latent_, up(a.q_rank, 64));
      ld_q_heads_ = std::max(ld_q_heads_, up(a.heads * up(a.dim, 16), 64));
      if (packs(a)) ld_packed_ = std::max(ld_packed_, up(a.heads * (up(a.dim, 16) + up(a.vdim, 16)), 64));
      max_absorbed_ = std::max(max_absorbed_, a.heads * g.k_dim);
      max_latent_k_ = std::max(max_latent_k_, g.k_dim);
    } else if (l.mixer == MixerKind::Retention) {
      const RetentionSpec& r = l.ret;
      RecurrentLayerGeometry g;
      g.width = r.heads * r.dim * r.vdim;
      rec_layers_.push_back(g);
      ld_proj_ = std::max(ld_proj_, up(2 * r.heads * (r.dim + r.vdim), 64));
      ld_mixer_ = std::max(ld_mixer_, up(r.heads * r.vdim, 64));
      max_rec_o_ = std::max(max_rec_o_, r.heads * r.vdim);
      qk_bytes_per_token_ = std::max(qk_bytes_per_token_, q38_retention_qk_bytes(1, r.heads, r.dim, act_));
    } else {
      RecurrentLayerGeometry g;
      g.width = l.rec.width;
      g.taps = l.mixer == MixerKind::RgLru ? l.rec.taps : 0;
      g.channels = g.taps ? l.rec.width : 0;
      rec_layers_.push_back(g);
      const int parts = l.mixer == MixerKind::MinGru ? 3 : 2;
      ld_proj_ = std::max(ld_proj_, up(parts * l.rec.width, 64));
      ld_mixer_ = std::max(ld_mixer_, up(l.rec.width, 64));
      if (l.mixer == MixerKind::RgLru) max_rec_ = std::max(max_rec_, l.rec.width);
    }
    if (l.ff) ld_ff_ = std::max(ld_ff_, up(l.ff, 64));
  }
  max_v_ = v_first;
  visit_weights(nullptr);
}

// ---- weights ----------------------------------------------------------------------------------------------
template <typename T>
const T* LayerListModel::put(DeviceArena* arena, const std::vector<T>& v) {
  const size_t bytes = up256(std::max<size_t>(v.size() * sizeof(T), 1));
  if (!arena) {
    weight_bytes_ += bytes;
    return nullptr;
  }
  void* dst = arena->allocate(bytes);
  QWEN38_CUDA(cudaMemcpy(dst, v.data(), v.size() * sizeof(T), cudaMemcpyHostToDevice));
  return static_cast<const T*>(dst);
}

const float* LayerListModel::put_f32(DeviceArena* arena, const std::string& name) {
  const TensorInfo& t = reader_.file().tensor(name);
  std::vector<float> v(size_t(t.numel()));
  if (arena)
    for (size_t i = 0; i < v.size(); ++i) v[i] = reader_.at(t, int64_t(i));
  return put(arena, v);
}

const q38_bf16* LayerListModel::put_bf16(DeviceArena* arena, const std::string& name) {
  const TensorInfo& t = reader_.file().tensor(name);
  std::vector<q38_bf16> v(size_t(t.numel()));
  if (arena) reader_.copy_bf16(t, 0, t.numel(), v.data());
  return put(arena, v);
}

// Stacks matrices [n_i][k] along n (or alternates the rows of two), rows padded with zeros to a multiple of 64 columns
// and the stack to a multiple of 16 rows.
kernels::DenseWeight LayerListModel::put_linear(DeviceArena* arena, const Linear& l) {
  kernels::DenseWeight d{};
  bool bias = false;
  for (size_t i = 0; i < l.weights.size(); ++i) {
    const TensorInfo& t = reader_.file().tensor(l.weights[i]);
    QWEN38_CHECK(t.shape.size() == 2 && (i == 0 || int(t.shape[1]) == d.k), l.weights[i], ": shape");
    d.n += l.heads_of.empty() ? int(t.shape[0]) : int(t.shape[0]) / l.heads_of[i] * up(l.heads_of[i], 16);
    d.k = int(t.shape[1]);
    bias = bias || !l.biases[i].empty();
  }
  d.ld = up(d.k, 64);
  std::vector<q38_bf16> w(size_t(up(d.n, 16)) * size_t(d.ld), 0);
  std::vector<float> b(bias ? size_t(up(d.n, 16)) : 0, 0.0f);
  if (arena) {
    int row0 = 0;
    for (size_t i = 0; i < l.weights.size(); ++i) {
      const TensorInfo& t = reader_.file().tensor(l.weights[i]);
      for (int64_t r = 0; r < t.shape[0]; ++r) {
        const int64_t in_head = l.heads_of.empty() ? r : r / l.heads_of[i] * up(l.heads_of[i], 16) + r % l.heads_of[i];
        const int64_t to = l.interleave ? 2 * r + int64_t(i) : row0 + in_head;
        reader_.copy_bf16(t, r * t.shape[1], t.shape[1], w.data() + to * d.ld);
        if (!l.biases[i].empty()) b[size_t(to)] = reader_.at(reader_.file().tensor(l.biases[i]), r);
      }
      row0 += l.heads_of.empty() ? int(t.shape[0]) : int(t.shape[0]) / l.heads_of[i] * up(l.heads_of[i], 16);
    }
  }
  d.w = put(arena, w);
  d.bias = bias ? put(arena, b) : nullptr;
  return d;
}

// One matrix [n_to][k] per head, rows padded to 64 columns: `name` holds the heads' rows one after the other,
// [heads * rows][cols]; with `transpose` a head's matrix is [cols][rows].
kernels::DenseWeight LayerListModel::put_heads(DeviceArena* arena, const std::string& name, int heads, int n_to, bool transpose) {
  const TensorInfo& t = reader_.file().tensor(name);
  const int rows = int(t.shape[0]) / heads, cols = int(t.shape[1]);
  kernels::DenseWeight d{};
  d.n = n_to;
  d.k = transpose ? rows : cols;
  d.ld = up(d.k, 64);
  std::vector<q38_bf16> w(size_t(up(heads * d.n, 16)) * size_t(d.ld), 0);
  if (arena) {
    std::vector<q38_bf16> line(size_t(cols), 0);
    for (int h = 0; h < heads; ++h)
      for (int r = 0; r < rows; ++r) {
        reader_.copy_bf16(t, (int64_t(h) * rows + r) * cols, cols, line.data());
        for (int c = 0; c < cols; ++c)
          w[transpose ? (size_t(h) * d.n + size_t(c)) * d.ld + size_t(r) : (size_t(h) * d.n + size_t(r)) * d.ld + size_t(c)] = line[size_t(c)];
      }
  }
  d.w = put(arena, w);
  return d;
}

StreamWeights LayerListModel::put_streams(DeviceArena* arena, int layer, const char* name) {
  const std::string p = at_layer(layer, name);
  if (hyper_) return {put_f32(arena, p + ".in"), put_f32(arena, p + ".out"), put_f32(arena, p + ".mix")};
  const float* one = put(arena, std::vector<float>{1.0f});
  return {one, one, one};
}

void LayerListModel::visit_weights(DeviceArena* arena) {
  weight_bytes_ = arena ? weight_bytes_ : 0;
  layers_.assign(cfg_.layers.size(), {});
  embed_ = put_bf16(arena, "embed");
  if (cfg_.learned_positions) pos_ = put_bf16(arena, "pos");
  for (int i = 0; i < cfg_.num_layers; ++i) {
    const LayerSpec& l = cfg_.layers[size_t(i)];
    LayerWeightsDev& W = layers_[size_t(i)];
    const LayerTensors names = names_of(l, i, design_.feed_forward);
    W.in = put_linear(arena, names.in);
    W.out = put_linear(arena, names.out);
    W.norm1 = put_f32(arena, at_layer(i, "norm1"));
    if (design_.post_norms) W.norm1b = put_f32(arena, at_layer(i, "norm1b"));
    else W.hc1 = put_streams(arena, i, "hc1");
    if (l.ff) {
      W.norm2 = put_f32(arena, at_layer(i, "norm2"));
      if (design_.post_norms) W.norm2b = put_f32(arena, at_layer(i, "norm2b"));
      else W.hc2 = put_streams(arena, i, "hc2");
      W.up = put_linear(arena, names.up);
      W.down = put_linear(arena, names.down);
      if (design_.feed_forward == LayerListDesign::FeedForward::Xielu) {
        const TensorInfo& t = reader_.file().tensor(at_layer(i, "mlp.act"));
        auto softplus = [](double x) { return std::max(x, 0.0) + std::log1p(std::exp(-std::abs(x))); };
        W.alpha_p = float(softplus(reader_.at(t, 0)));
        W.alpha_n = float(0.5 + softplus(reader_.at(t, 1)));
      }
    }
    if (l.mixer == MixerKind::Retention) {
      const RetentionSpec& r = l.ret;
      std::vector<double> freq(size_t(r.rot_dims / 2));
      for (size_t k = 0; k < freq.size(); ++k) freq[k] = std::pow(r.rot_base, -2.0 * double(k) / double(r.rot_dims));
      W.inv_freq = put(arena, freq);
      std::vector<float> pow_table;
      for (const double d : r.decay)
        for (int k = 0; k <= Q38_RETENTION_CHUNK; ++k) pow_table.push_back(float(std::pow(d, double(k))));
      W.decay_pow = put(arena, pow_table);
    }
    if (l.mixer == MixerKind::LatentAttention) {
      const LatentAttentionSpec& a = l.latent;
      W.q_gain = put_f32(arena, mix(i, "dq.norm"));
      W.kv_gain = put_f32(arena, mix(i, "dkv.norm"));
      W.uq = put_linear(arena, {{mix(i, "uq")}, {""}, false, {a.dim}});
      W.uk = put_heads(arena, mix(i, "uk"), a.heads, up(a.kv_rank, 32), true);
      W.uv = put_heads(arena, mix(i, "uv"), a.heads, a.vdim, false);
      if (packs(a)) W.ukv = put_linear(arena, {{mix(i, "uk"), mix(i, "uv")}, {"", ""}, false, {a.dim, a.vdim}});
    }
    if (l.mixer == MixerKind::Attention) {
      if (l.attn.value_mix) W.v_mix = put_f32(arena, mix(i, "vmix"));
      std::vector<double> freq(size_t(l.attn.rot_dims / 2));
      for (size_t k = 0; k < freq.size(); ++k) freq[k] = std::pow(l.attn.rot_base, -2.0 * double(k) / double(l.attn.rot_dims));
      W.inv_freq = put(arena, freq);
      if (l.attn.head_mix) W.head_mix = put_f32(arena, mix(i, "talk"));
    }
    if (l.mixer == MixerKind::RgLru) {
      const int width = l.rec.width, blocks = l.rec.blocks, bs = width / blocks, taps = l.rec.taps;
      W.block_ld = up(bs, 32);
      std::vector<float> conv(size_t(taps) * size_t(width)), gate_b(size_t(2) * size_t(width));
      std::vector<q38_bf16> gates(size_t(blocks) * 2 * size_t(W.block_ld) * size_t(W.block_ld), 0);
      if (arena) {
        const TensorInfo& ct = reader_.file().tensor(mix(i, "conv"));
        for (int c = 0; c < width; ++c)
          for (int j = 0; j < taps; ++j) conv[size_t(j) * width + c] = reader_.at(ct, int64_t(c) * taps + j);
        for (int g = 0; g < 2; ++g) {
          const TensorInfo& gt = reader_.file().tensor(mix(i, g ? "ri" : "ra"));
          const TensorInfo& bt = reader_.file().tensor(mix(i, g ? "ri.b" : "ra.b"));
          for (int c = 0; c < width; ++c) gate_b[size_t(g) * width + c] = reader_.at(bt, c);
          for (int b = 0; b < blocks; ++b)
            for (int o = 0; o < bs; ++o)
              reader_.copy_bf16(gt, (int64_t(b) * bs + o) * bs, bs, gates.data() + ((size_t(b) * 2 + g) * W.block_ld + o) * W.block_ld);
        }
      }
      W.conv_w = put(arena, conv);
      W.conv_b = put_f32(arena, mix(i, "conv.b"));
      W.gate_w = put(arena, gates);
      W.gate_b = put(arena, gate_b);
      W.lam = put_f32(arena, mix(i, "lam"));
    }
  }
  final_norm_ = put_f32(arena, "final.norm");
  ones_ = put(arena, std::vector<float>(size_t(streams_), 1.0f));
  head_ = put_linear(arena, {{"head"}, {""}});
}

void LayerListModel::load_weights() {
  arena_ = DeviceArena(weight_bytes_ + 256);
  visit_weights(&arena_);
}

// ---- activations -------------------------------------------------------------------------------------------
void LayerListModel::carve(Workspace& w, const StepContext& ctx) {
  const size_t T = size_t(ctx.max_tokens), R = size_t(ctx.max_rows);
  const size_t gemm_partials = f32_ ? 0 : size_t(2) * size_t(ctx.num_sms) * 128 * 256;
  residual_ = w.take<float>(T * size_t(streams_) * size_t(cfg_.hidden_size));
  x_ = w.take<uint8_t>(T * size_t(ld_x_) * elem_);
  proj_ = w.take<uint8_t>(T * size_t(ld_proj_) * elem_);
  mixer_ = w.take<uint8_t>(T * size_t(ld_mixer_) * elem_);
  ff_ = w.take<uint8_t>(T * size_t(ld_ff_) * elem_);
  y_ = w.take<float>(T * size_t(ld_x_));
  q_ = w.take<uint8_t>(T * size_t(max_q_) * elem_);
  v_first_ = w.take<uint8_t>(T * size_t(max_v_) * elem_);
  stats_ = w.take<float>(T * size_t(max_heads_) * 2 * kStatSplits);
  if (!f32_) partials_ = w.take<float>(R * kMaxSplits * (size_t(max_attn_out_) + 2 * size_t(max_heads_)));
  rec_scratch_ = w.take<float>(2 * T * size_t(max_rec_));
  qk_ = w.take<uint8_t>(T * qk_bytes_per_token_);
  rec_o_ = w.take<float>(T * size_t(max_rec_o_));
  q_latent_ = w.take<uint8_t>(T * size_t(ld_q_latent_) * elem_);
  q_heads_ = w.take<uint8_t>(T * size_t(ld_q_heads_) * elem_);
  q_absorbed_ = w.take<uint8_t>(T * size_t(max_absorbed_) * elem_);
  o_latent_ = w.take<uint8_t>(T * size_t(max_absorbed_) * elem_);
  latent_partial_floats_ = f32_ || !max_latent_k_ ? 0 : q38_latent_attention_partial_floats(max_latent_k_);
  latent_partials_ = w.take<float>(latent_partial_floats_);
  if (ld_packed_) {
    // several chunks' worth of context, at most 1 GiB, no more than all slots can hold; longer contexts stay in latent form
    const int64_t bytes = (int64_t(ld_packed_) + max_latent_k_) * 2;
    packed_rows_ = std::min<int64_t>(std::max<int64_t>(8 * int64_t(T), 16384), (int64_t(1) << 30) / bytes);
    packed_rows_ = std::min<int64_t>(packed_rows_, int64_t(R) * up(max_context_, 64)) / 64 * 64;
    packed_latents_ = w.take<uint8_t>(size_t(packed_rows_) * size_t(max_latent_k_) * 2);
    packed_kv_ = w.take<uint8_t>(size_t(packed_rows_) * size_t(ld_packed_) * 2);
  }
  head_x_ = w.take<uint8_t>(R * size_t(ld_x_) * elem_);
  gemm_ws_.partials = w.take<float>(gemm_partials);
  gemm_ws_.partial_floats = gemm_partials;
  gemm_ws_.counters = w.take<int>(4096);
  gemm_ws_.num_counters = 4096;
}

void LayerListModel::prepare(const StepContext& ctx) {
  if (score_heads_ > 0)
    scores_ = DeviceBuffer(size_t(ctx.kv->num_pages()) * size_t(score_heads_) * kernels::kPageTokens * 4);
}

// ---- the step ------------------------------------------------------------------------------------------------
void LayerListModel::attention(const StepContext& ctx, const StepBatch& b, const LayerSpec& l, const LayerWeightsDev& W,
                               int attn_i, bool first_values, bool blend) {
  const AttentionSpec& a = l.attn;
  const kernels::KvLayerDesc kv = ctx.kv->layer_desc(attn_i);
  kernels::RopeAppendParams rp{};
  rp.proj = proj_;
  rp.ld_proj = ld_proj_;
  rp.act = act_;
  rp.heads = a.heads;
  rp.kv_heads = a.kv_heads;
  rp.dim = a.dim;
  rp.vdim = a.vdim;
  rp.rot_dims = a.rot_dims;
  rp.inv_freq = W.inv_freq;
  rp.q_out = q_;
  rp.v_first_out = first_values ? v_first_ : nullptr;
  rp.v_first_in = blend ? v_first_ : nullptr;
  rp.v_mix = W.v_mix;
  kernels::rope_append(rp, b.all, kv, ctx.stream);
  ctx.mark("mix.rope_append");
  kernels::MixedAttentionParams ap{};
  ap.q = q_;
  ap.act = act_;
  ap.heads = a.heads;
  ap.vdim = a.vdim;
  ap.scale = a.scale;
  ap.head_mix = W.head_mix;
  ap.out = mixer_;
  ap.ld_out = ld_mixer_;
  ap.stats = stats_;
  ap.stat_splits = kStatSplits;
  ap.scores = scores_.as<float>();
  ap.partials = partials_;
  ap.max_splits = kMaxSplits;
  if (b.decode || b.mixed) kernels::mixed_attention_decode(ap, b.single_part, kv, ctx.stream);
  if (!b.decode) kernels::mixed_attention_prefill(ap, b.chunk_part, kv, ctx.stream);
  ctx.mark(b.decode ? "mix.attn_decode" : "mix.attn_prefill");
}

// In the latent space a (query, key) pair costs 2 kv_rank multiplications per head (half of them twice, for the weights'
// second term), with keys and values of their own dim + vdim; those have to be made from every latent of the contexts first,
// by a product that runs at a few times the attention kernels' rate.
bool LayerListModel::packing_pays(const LatentAttentionSpec& a, const StepBatch& b) const {
  if (b.decode || !packs(a) || b.chunk_packed_rows > packed_rows_ || b.chunk_part.num_seqs == 0) return false;
  const double per_seq = double(b.chunk_part.num_tokens) / b.chunk_part.num_seqs, own = a.dim + a.vdim;
  return per_seq * 1.5 * (2.0 * a.kv_rank - own) > 0.5 * a.kv_rank * own;
}

void LayerListModel::latent_attention(const StepContext& ctx, const StepBatch& b, const LayerSpec& l, const LayerWeightsDev& W, int attn_i) {
  const LatentAttentionSpec& a = l.latent;
  const kernels::KvLayerDesc kv = ctx.kv->layer_desc(attn_i);
  const int k_ld = up(a.dim, 16), v_ld = up(a.vdim, 16);
  const uint8_t* gate = proj_ + size_t(a.q_rank + a.kv_rank) * elem_;
  kernels::LatentAppendParams lp{};
  lp.proj = proj_;
  lp.ld_proj = ld_proj_;
  lp.act = act_;
  lp.q_rank = a.q_rank;
  lp.kv_rank = a.kv_rank;
  lp.q_gain = W.q_gain;
  lp.kv_gain = W.kv_gain;
  lp.eps = cfg_.rms_norm_eps;
  lp.q_out = q_latent_;
  lp.ld_q = ld_q_latent_;
  kernels::latent_append(lp, b.all, kv, ctx.stream);
  ctx.mark("mix.latent_append");
  gemm(ctx, q_latent_, ld_q_latent_, b.m, W.uq, Q38_DENSE_STORE, q_heads_, ld_q_heads_);
  ctx.mark("gemm.latent_uq");
  int first = 0;  // rows from here on are served in the latent space
  if (packing_pays(a, b)) {
    first = b.chunk_part.num_tokens;
    const int rows = int(b.chunk_packed_rows);
    kernels::latent_gather(b.chunk_part, kv, b.chunk_longest_context, rows, packed_latents_, ctx.stream);
    ctx.mark("mix.latent_gather");
    gemm(ctx, packed_latents_, kv.k_dim, rows, W.ukv, Q38_DENSE_STORE, packed_kv_, ld_packed_);
    ctx.mark("gemm.latent_kv");
    kernels::PackedAttentionParams pp{};
    pp.q = q_heads_;
    pp.ld_q = ld_q_heads_;
    pp.q_stride = k_ld;
    pp.k = packed_kv_;
    pp.v = packed_kv_ + size_t(a.heads) * size_t(k_ld) * 2;
    pp.ld_kv = ld_packed_;
    pp.k_stride = k_ld;
    pp.v_stride = v_ld;
    pp.heads = a.heads;
    pp.dim = a.dim;
    pp.vdim = a.vdim;
    pp.scale = a.scale;
    pp.gate = gate;
    pp.ld_gate = ld_proj_;
    pp.out = mixer_;
    pp.ld_out = ld_mixer_;
    kernels::packed_attention(pp, b.chunk_part, ctx.stream);
    ctx.mark("mix.latent_prefill");
  }
  const int rows = b.m - first;
  if (rows == 0) return;
  const auto row = [&](uint8_t* base, int ld) { return base + size_t(first) * size_t(ld) * elem_; };
  const int ld_k = a.heads * kv.k_dim;
  kernels::DenseEpilogue ep{};
  ep.kind = Q38_DENSE_STORE;
  ep.out = row(q_absorbed_, ld_k);
  ep.ldo = ld_k;
  kernels::dense_gemm_grouped(row(q_heads_, ld_q_heads_), ld_q_heads_, act_, rows, W.uk, {a.heads, k_ld, kv.k_dim}, ep, gemm_ws_, ctx.stream);
  ctx.mark("gemm.latent_uk");
  kernels::LatentAttentionParams ap{};
  ap.q = q_absorbed_;
  ap.act = act_;
  ap.heads = a.heads;
  ap.scale = a.scale;
  ap.out = o_latent_;
  ap.partials = latent_partials_;
  ap.partial_floats = latent_partial_floats_;
  if (b.decode || b.mixed) kernels::latent_attention(ap, b.single_part, kv, ctx.stream);
  if (!b.decode && first == 0) kernels::latent_attention(ap, b.chunk_part, kv, ctx.stream);
  ctx.mark(b.decode ? "mix.latent_decode" : "mix.latent_prefill");
  ep.kind = Q38_DENSE_GATE_SIGMOID;
  ep.out = row(mixer_, ld_mixer_);
  ep.ldo = ld_mixer_;
  ep.gate = gate + size_t(first) * size_t(ld_proj_) * elem_;
  ep.ld_gate = ld_proj_;
  kernels::dense_gemm_grouped(row(o_latent_, ld_k), ld_k, act_, rows, W.uv, {a.heads, kv.k_dim, a.vdim}, ep, gemm_ws_, ctx.stream);
  ctx.mark("gemm.latent_uv");
}

void LayerListModel::retention(const StepContext& ctx, const StepBatch& b, const LayerSpec& l, const LayerWeightsDev& W,
                               const kernels::RecurrentStateDesc& st) {
  const RetentionSpec& r = l.ret;
  kernels::RetentionParams p{};
  p.proj = proj_;
  p.ld_proj = ld_proj_;
  p.act = act_;
  p.heads = r.heads;
  p.dim = r.dim;
  p.vdim = r.vdim;
  p.rot_dims = r.rot_dims;
  p.inv_freq = W.inv_freq;
  p.decay_pow = W.decay_pow;
  p.k_scale = float(1.0 / std::sqrt(double(r.dim)));
  p.eps = cfg_.rms_norm_eps;
  p.qk = qk_;
  p.o = rec_o_;
  p.out = mixer_;
  p.ld_out = ld_mixer_;
  if (b.decode || b.mixed) kernels::retention(p, b.single_part, st, ctx.stream);
  if (!b.decode) kernels::retention(p, b.chunk_part, st, ctx.stream);
  ctx.mark("mix.retention");
}

void LayerListModel::recurrent(const StepContext& ctx, const StepBatch& b, const LayerSpec& l, const LayerWeightsDev& W, int rec_i) {
  const kernels::RecurrentStateDesc st = state_->layer_desc(rec_i);
  if (l.mixer == MixerKind::Retention) return retention(ctx, b, l, W, st);
  if (l.mixer == MixerKind::MinGru) {
    const kernels::MinGruParams p{proj_, ld_proj_, act_, l.rec.width, mixer_, ld_mixer_};
    if (b.decode || b.mixed) kernels::mingru(p, b.single_part, st, ctx.stream);
    if (!b.decode) kernels::mingru(p, b.chunk_part, st, ctx.stream);
    ctx.mark("mix.mingru");
    return;
  }
  kernels::RgLruParams p{};
  p.proj = proj_;
  p.ld_proj = ld_proj_;
  p.act = act_;
  p.width = l.rec.width;
  p.blocks = l.rec.blocks;
  p.block_ld = W.block_ld;
  p.taps = l.rec.taps;
  p.conv_w = W.conv_w;
  p.conv_b = W.conv_b;
  p.gate_w = W.gate_w;
  p.gate_b = W.gate_b;
  p.lam = W.lam;
  p.log_decay = design_.rglru_log_decay;
  p.scratch = rec_scratch_;
  p.out = mixer_;
  p.ld_out = ld_mixer_;
  if (b.decode || b.mixed) kernels::rglru(p, b.single_part, st, ctx.stream);
  if (!b.decode) kernels::rglru(p, b.chunk_part, st, ctx.stream);
  ctx.mark("mix.rglru");
}

void LayerListModel::join_residual(const StepContext& ctx, int m, const Sublayer& done, const Sublayer& next) {
  const kernels::Norm pre = norm(next.pre);
  const kernels::Norm* then = next.pre ? &pre : nullptr;
  if (design_.post_norms)
    kernels::residual_norm(y_, ld_x_, m, cfg_.hidden_size, norm(done.post), residual_, then, x_, ld_x_, act_, ctx.stream);
  else
    kernels::stream_norm(y_, ld_x_, m, cfg_.hidden_size, streams_, {done.hc.mix, done.hc.out, cfg_.residual_mult}, residual_,
                         next.hc.in, then, x_, ld_x_, act_, ctx.stream);
  ctx.mark("residual_norm");
}

void LayerListModel::feed_forward(const StepContext& ctx, int m, const LayerWeightsDev& W) {
  kernels::DenseEpilogue ep{};
  ep.out = ff_;
  ep.ldo = ld_ff_;
  ep.alpha_p = W.alpha_p;
  ep.alpha_n = W.alpha_n;
  switch (design_.feed_forward) {
    case LayerListDesign::FeedForward::GeluGlu: ep.kind = Q38_DENSE_GLU_GELU; break;
    case LayerListDesign::FeedForward::SiluGlu: ep.kind = Q38_DENSE_GLU_SILU; break;
    case LayerListDesign::FeedForward::Xielu: ep.kind = Q38_DENSE_XIELU; break;
  }
  kernels::dense_gemm(x_, ld_x_, act_, m, W.up, ep, gemm_ws_, ctx.stream);
  ctx.mark(design_.feed_forward == LayerListDesign::FeedForward::Xielu ? "gemm.mlp_up" : "gemm.mlp_gate_up");
  gemm(ctx, ff_, ld_ff_, m, W.down, Q38_DENSE_STORE_F32, y_, ld_x_);
  ctx.mark("gemm.mlp_down");
}

void LayerListModel::forward(const StepContext& ctx, const StepBatch& b) {
  constexpr const char* kIn[] = {"gemm.attn_qkv", "gemm.mingru_in", "gemm.rglru_in", "gemm.retention_in", "gemm.latent_in"};
  constexpr const char* kOut[] = {"gemm.attn_o", "gemm.mingru_out", "gemm.rglru_out", "gemm.retention_out", "gemm.latent_o"};
  const int m = b.m, H = cfg_.hidden_size, n = int(runs_.size());
  const Sublayer nothing;
  if (design_.post_norms) {
    kernels::embed_norm(embed_, pos_, b.tokens, b.all.tok_pos, m, H, residual_, norm(n ? mixer_of(0).pre : final_norm_), x_, ld_x_, act_,
                        ctx.stream);
  } else {
    kernels::stream_embed(embed_, b.tokens, m, H, cfg_.embedding_scale, streams_, residual_, n ? mixer_of(0).hc.in : ones_,
                          norm(n ? mixer_of(0).pre : final_norm_), x_, ld_x_, act_, ctx.stream);
  }
  ctx.mark("embed");
  int attn_i = 0, rec_i = 0;
  bool have_values = false;
  for (int i = 0; i < n; ++i) {
    const LayerSpec& l = cfg_.layers[size_t(runs_[size_t(i)])];
    const LayerWeightsDev& W = layers_[size_t(runs_[size_t(i)])];
    // what follows this run; the last one's successor is the final norm, taken over the sampled rows only
    const Sublayer next = i + 1 < n ? mixer_of(i + 1) : nothing;
    gemm(ctx, x_, ld_x_, m, W.in, Q38_DENSE_STORE, proj_, ld_proj_);
    ctx.mark(kIn[int(l.mixer)]);
    if (l.mixer == MixerKind::Attention) {
      attention(ctx, b, l, W, attn_i++, l.attn.value_mix && !have_values, l.attn.value_mix && have_values);
      have_values = have_values || l.attn.value_mix;
    } else if (l.mixer == MixerKind::LatentAttention) {
      latent_attention(ctx, b, l, W, attn_i++);
    } else {
      recurrent(ctx, b, l, W, rec_i++);
    }
    gemm(ctx, mixer_, ld_mixer_, m, W.out, Q38_DENSE_STORE_F32, y_, ld_x_);
    ctx.mark(kOut[int(l.mixer)]);
    join_residual(ctx, m, mixer_of(i), l.ff ? feed_forward_of(i) : next);
    if (!l.ff) continue;
    feed_forward(ctx, m, W);
    join_residual(ctx, m, feed_forward_of(i), next);
  }
}

void LayerListModel::head(const StepContext& ctx, const HeadRows& rows, float* logits) {
  if (design_.post_norms)
    kernels::gather_norm(residual_, rows.rows, rows.first, rows.count, cfg_.hidden_size, norm(final_norm_), head_x_, ld_x_, act_, ctx.stream);
  else
    kernels::stream_gather(residual_, rows.rows, rows.first, rows.count, cfg_.hidden_size, streams_, norm(final_norm_), head_x_, ld_x_,
                           act_, ctx.stream);
  gemm(ctx, head_x_, ld_x_, rows.count, head_, Q38_DENSE_STORE_F32, logits, cfg_.vocab_size);
  ctx.mark("gemm.lm_head");
}

}  // namespace

std::unique_ptr<StepModel> make_layer_list_model(const ModelFile& file, const RunnerOptions& options,
                                                 const LayerListDesign& design) {
  return std::make_unique<LayerListModel>(file, options, design);
}

void check_layer_list_tensors(const ModelFile& file, const LayerListDesign& design) {
  const ModelConfig& c = file.config();
  const TensorReader r(file);
  const int64_t W = c.hidden_size, V = c.vocab_size;
  const std::vector<int64_t> gain = design.norm_gain_is_scalar ? std::vector<int64_t>{} : std::vector<int64_t>{W};
  r.require("embed", {V, W});
  if (c.learned_positions) r.require("pos", {c.max_position_embeddings, W});
  r.require("final.norm", gain);
  r.require("head", {V, W});
  for (int i = 0; i < c.num_layers; ++i) {
    const LayerSpec& l = c.layers[size_t(i)];
    auto linear = [&](const char* name, int64_t n, int64_t k, bool bias) {
      r.require(mix(i, name), {n, k});
      if (bias) r.require(mix(i, (std::string(name) + ".b").c_str()), {n});
    };
    const int64_t S = c.streams;
    auto streams = [&](const char* name) {
      if (S == 0 || (S == 1 && !file.has_tensor(at_layer(0, "hc1.in")))) return;
      const std::string p = at_layer(i, name);
      r.require(p + ".in", {S});
      r.require(p + ".out", {S});
      r.require(p + ".mix", {S, S});
    };
    const bool xielu = design.feed_forward == LayerListDesign::FeedForward::Xielu;
    r.require(at_layer(i, "norm1"), gain);
    if (design.post_norms) r.require(at_layer(i, "norm1b"), gain);
    streams("hc1");
    if (l.ff) {
      r.require(at_layer(i, "norm2"), gain);
      if (design.post_norms) r.require(at_layer(i, "norm2b"), gain);
      streams("hc2");
      if (xielu) r.require(at_layer(i, "mlp.act"), {2});
      else r.require(at_layer(i, "mlp.gate"), {l.ff, W});
      r.require(at_layer(i, "mlp.up"), {l.ff, W});
      r.require(at_layer(i, "mlp.down"), {W, l.ff});
    }
    if (l.mixer == MixerKind::Attention) {
      const AttentionSpec& a = l.attn;
      linear("q", int64_t(a.heads) * a.dim, W, true);
      linear("k", int64_t(a.kv_heads) * a.dim, W, true);
      linear("v", int64_t(a.kv_heads) * a.vdim, W, true);
      linear("o", W, int64_t(a.heads) * a.vdim, true);
      if (a.head_mix) r.require(mix(i, "talk"), {a.heads, a.heads});
      if (a.value_mix) r.require(mix(i, "vmix"), {});
    } else if (l.mixer == MixerKind::MinGru) {
      linear("z", l.rec.width, W, true);
      linear("x", l.rec.width, W, true);
      linear("g", l.rec.width, W, false);
      linear("o", W, l.rec.width, false);
    } else if (l.mixer == MixerKind::Retention) {
      const RetentionSpec& t = l.ret;
      linear("q", int64_t(t.heads) * t.dim, W, false);
      linear("k", int64_t(t.heads) * t.dim, W, false);
      linear("v", int64_t(t.heads) * t.vdim, W, false);
      linear("g", int64_t(t.heads) * t.vdim, W, false);
      linear("o", W, int64_t(t.heads) * t.vdim, false);
    } else if (l.mixer == MixerKind::LatentAttention) {
      const LatentAttentionSpec& a = l.latent;
      linear("dq", a.q_rank, W, false);
      r.require(mix(i, "dq.norm"), {a.q_rank});
      linear("uq", int64_t(a.heads) * a.dim, a.q_rank, false);
      linear("dkv", a.kv_rank, W, false);
      r.require(mix(i, "dkv.norm"), {a.kv_rank});
      linear("uk", int64_t(a.heads) * a.dim, a.kv_rank, false);
      linear("uv", int64_t(a.heads) * a.vdim, a.kv_rank, false);
      linear("g", int64_t(a.heads) * a.vdim, W, false);
      linear("o", W, int64_t(a.heads) * a.vdim, false);
    } else {
      const int64_t w = l.rec.width, nb = l.rec.blocks, bs = w / nb;
      linear("y", w, W, true);
      linear("x", w, W, true);
      r.require(mix(i, "conv"), {w, l.rec.taps});
      r.require(mix(i, "conv.b"), {w});
      for (const char* g : {"ra", "ri"}) {
        r.require(mix(i, g), {nb, bs, bs});
        r.require(mix(i, (std::string(g) + ".b").c_str()), {nb, bs});
      }
      r.require(mix(i, "lam"), {w});
      linear("o", W, w, false);
    }
  }
}

}  // namespace qwen38
