// The Nololix design: config.json reader and conventions. Layers of two kinds (retention, latent attention with an output
// gate), pre-norms over equal parts of the row, residual streams joined by hyper-connections, an ungated xIELU feed-forward
// where the configuration lists one, and a span of layers that runs several times with the same weights.
#include "layer_list_model.h"

namespace qwen38 {

namespace {

LayerListDesign nololix_design() {
  LayerListDesign d;
  d.feed_forward = LayerListDesign::FeedForward::Xielu;
  d.norm_gain_is_scalar = false;
  d.post_norms = false;
  return d;
}

bool given(const jsonmin::Value& j, const char* key) {
  const jsonmin::Value* v = j.find(key);
  return v && v->kind != jsonmin::Value::Null;
}

ModelConfig read_nololix(const jsonmin::Value& j) {
  ModelConfig c;
  c.hidden_size = int(j.at("width").as_int());
  c.vocab_size = int(j.at("vocab").as_int());
  c.max_position_embeddings = 1 << 24;  // nothing in the design bounds the context
  c.rms_norm_eps = float(j.at("norm").at("eps").as_double());
  c.norm_groups = given(j.at("norm"), "groups") ? int(j.at("norm").at("groups").as_int()) : 1;
  c.embedding_scale = given(j, "embedding") && given(j.at("embedding"), "scale") ? float(j.at("embedding").at("scale").as_double()) : 1.0f;
  c.residual_mult = given(j, "residual_mult") ? float(j.at("residual_mult").as_double()) : 1.0f;
  c.streams = given(j, "streams") ? int(j.at("streams").as_int()) : 0;
  QWEN38_CHECK(c.hidden_size > 0 && c.vocab_size > 0, "width and vocab must be positive");
  QWEN38_CHECK(c.norm_groups > 0 && c.hidden_size % c.norm_groups == 0, c.norm_groups, " norm groups of a width of ", c.hidden_size);
  QWEN38_CHECK(c.streams >= 0 && c.streams <= Q38_MAX_STREAMS, c.streams, " residual streams (at most ", Q38_MAX_STREAMS, ")");
  int index = 0;
  for (const jsonmin::Value& layer : j.at("layers").arr) {
    LayerSpec l;
    const std::string where = "layer " + std::to_string(index++);
    const std::string& type = layer.at("type").as_string();
    const jsonmin::Value& m = layer.at("mixer");
    if (type == "retention") {
      l.mixer = MixerKind::Retention;
      RetentionSpec& r = l.ret;
      r.heads = int(m.at("heads").as_int());
      r.dim = int(m.at("dim").as_int());
      r.vdim = int(m.at("vdim").as_int());
      if (given(m, "rot")) {
        r.rot_dims = int(m.at("rot").at("dims").as_int());
        r.rot_base = m.at("rot").at("base").as_double();
      }
      for (const jsonmin::Value& d : m.at("decay").arr) r.decay.push_back(d.as_double());
      QWEN38_CHECK(r.heads > 0 && r.dim > 0 && r.vdim > 0, where, ": sizes");
      QWEN38_CHECK(r.rot_dims >= 0 && r.rot_dims % 2 == 0 && r.rot_dims <= r.dim, where, ": ", r.rot_dims, " rotated dimensions of ", r.dim);
      QWEN38_CHECK(int(r.decay.size()) == r.heads, where, ": ", r.decay.size(), " decays for ", r.heads, " heads");
    } else if (type == "latent_attention") {
      l.mixer = MixerKind::LatentAttention;
      LatentAttentionSpec& a = l.latent;
      a.heads = int(m.at("heads").as_int());
      a.dim = int(m.at("dim").as_int());
      a.vdim = int(m.at("vdim").as_int());
      a.q_rank = int(m.at("q_rank").as_int());
      a.kv_rank = int(m.at("kv_rank").as_int());
      a.scale = float(m.at("scale").as_double());
      QWEN38_CHECK(a.heads > 0 && a.dim > 0 && a.vdim > 0 && a.q_rank > 0 && a.kv_rank > 0, where, ": sizes");
    } else {
      fail(where + ": mixer '" + type + "' is not part of this design");
    }
    const jsonmin::Value* mlp = layer.find("mlp");
    if (mlp && mlp->kind == jsonmin::Value::Object) {
      QWEN38_CHECK(mlp->at("kind").as_string() == "dense", where, ": feed-forward '", mlp->at("kind").as_string(), "' is not part of this design");
      l.ff = int(mlp->at("ff").as_int());
      QWEN38_CHECK(l.ff > 0, where, ": ff");
    }
    c.is_attention.push_back(l.mixer == MixerKind::LatentAttention);
    c.layers.push_back(l);
  }
  c.num_layers = int(c.layers.size());
  if (given(j, "loop")) {
    const jsonmin::Value& loop = j.at("loop");
    c.loop_start = int(loop.at("start").as_int());
    c.loop_stop = int(loop.at("stop").as_int());
    c.loop_times = int(loop.at("times").as_int());
    QWEN38_CHECK(c.loop_start >= 0 && c.loop_start <= c.loop_stop && c.loop_stop <= c.num_layers && c.loop_times >= 1, "loop over layers ",
                 c.loop_start, " .. ", c.loop_stop - 1, ", ", c.loop_times, " times, in a model of ", c.num_layers);
  }
  return c;
}

const ArchitectureRegistration registration{
    {"Nololix", &read_nololix, [](const ModelFile& f) { check_layer_list_tensors(f, nololix_design()); },
     [](const ModelFile& f, const RunnerOptions& o) -> std::unique_ptr<StepModel> {
       return make_layer_list_model(f, o, nololix_design());
     }}};

}  // namespace

}  // namespace qwen38
