// The Fegenex design: config.json reader and conventions. Layers of three kinds (attention with head-mixed weights and
// value blending, minGRU, RG-LRU), each sublayer between two RMS norms with a single gain, a gelu-gated feed-forward
// where the configuration lists one, learned positions added to the embedding.
#include "layer_list_model.h"

namespace qwen38 {

namespace {

LayerListDesign fegenex_design() {
  LayerListDesign d;
  d.feed_forward = LayerListDesign::FeedForward::GeluGlu;
  d.norm_gain_is_scalar = true;
  d.rglru_log_decay = -8.0f;
  return d;
}

ModelConfig read_fegenex(const jsonmin::Value& j) {
  ModelConfig c;
  c.hidden_size = int(j.at("width").as_int());
  c.vocab_size = int(j.at("vocab").as_int());
  c.max_position_embeddings = int(j.at("max_positions").as_int());
  c.learned_positions = true;
  c.rms_norm_eps = float(j.at("norm").at("eps").as_double());
  QWEN38_CHECK(c.hidden_size > 0 && c.vocab_size > 0 && c.max_position_embeddings > 0, "width, vocab and max_positions must be positive");
  int index = 0;
  for (const jsonmin::Value& layer : j.at("layers").arr) {
    LayerSpec l;
    const std::string where = "layer " + std::to_string(index++);
    const std::string& type = layer.at("type").as_string();
    const jsonmin::Value& m = layer.at("mixer");
    if (type == "attention") {
      l.mixer = MixerKind::Attention;
      AttentionSpec& a = l.attn;
      a.heads = int(m.at("heads").as_int());
      a.kv_heads = int(m.at("kv_heads").as_int());
      a.dim = int(m.at("dim").as_int());
      a.vdim = int(m.at("vdim").as_int());
      if (const jsonmin::Value* rot = m.find("rot"); rot && rot->kind == jsonmin::Value::Object) {
        a.rot_dims = int(rot->at("dims").as_int());
        a.rot_base = rot->at("base").as_double();
      }
      a.scale = float(m.at("scale").as_double());
      a.value_mix = m.has("v_mix") && m.at("v_mix").kind == jsonmin::Value::Bool && m.at("v_mix").b;
      a.head_mix = true;
      QWEN38_CHECK(a.heads > 0 && a.kv_heads > 0 && a.heads % a.kv_heads == 0, where, ": ", a.heads, " query heads over ", a.kv_heads);
      QWEN38_CHECK(a.dim > 0 && a.vdim > 0 && a.rot_dims >= 0 && a.rot_dims % 2 == 0 && a.rot_dims <= a.dim, where, ": head sizes");
    } else if (type == "mingru") {
      l.mixer = MixerKind::MinGru;
      l.rec.width = int(m.at("width").as_int());
      QWEN38_CHECK(l.rec.width > 0, where, ": width");
    } else if (type == "rglru") {
      l.mixer = MixerKind::RgLru;
      l.rec.width = int(m.at("width").as_int());
      l.rec.blocks = int(m.at("blocks").as_int());
      l.rec.taps = int(m.at("conv").as_int());
      QWEN38_CHECK(l.rec.width > 0 && l.rec.blocks > 0 && l.rec.width % l.rec.blocks == 0 && l.rec.taps > 0, where, ": sizes");
    } else {
      fail(where + ": mixer '" + type + "' is not part of this design");
    }
    const jsonmin::Value* mlp = layer.find("mlp");
    if (mlp && mlp->kind == jsonmin::Value::Object) {
      QWEN38_CHECK(mlp->at("kind").as_string() == "dense", where, ": feed-forward '", mlp->at("kind").as_string(), "' is not part of this design");
      l.ff = int(mlp->at("ff").as_int());
      QWEN38_CHECK(l.ff > 0, where, ": ff");
    }
    c.is_attention.push_back(l.mixer == MixerKind::Attention);
    c.layers.push_back(l);
  }
  c.num_layers = int(c.layers.size());
  return c;
}

const ArchitectureRegistration registration{
    {"Fegenex", &read_fegenex, [](const ModelFile& f) { check_layer_list_tensors(f, fegenex_design()); },
     [](const ModelFile& f, const RunnerOptions& o) -> std::unique_ptr<StepModel> {
       return make_layer_list_model(f, o, fegenex_design());
     }}};

}  // namespace

}  // namespace qwen38
