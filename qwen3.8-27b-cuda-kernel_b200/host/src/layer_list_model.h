// A decoder that runs the layers its configuration lists: per layer a sequence mixer (attention with mixed heads, minGRU,
// RG-LRU, retention, latent attention) and optionally a feed-forward. A sublayer stands between a pre-norm and a post-norm
// whose output joins the residual, or behind a pre-norm only, with one or several residual streams.
// Dense bf16 weights; activations bf16 or fp32. A design provides names and conventions (LayerListDesign); everything
// below - weights, cache, state, step - is shared by the designs.
#pragma once

#include "step_model.h"

namespace qwen38 {

struct LayerListDesign {
  enum class FeedForward { GeluGlu, SiluGlu, Xielu };
  FeedForward feed_forward = FeedForward::GeluGlu;
  bool norm_gain_is_scalar = true;
  bool post_norms = true;
  float rglru_log_decay = -8.0f;
};

std::unique_ptr<StepModel> make_layer_list_model(const ModelFile& file, const RunnerOptions& options,
                                                 const LayerListDesign& design);
// Names and shapes of every tensor the layers need; throws Error on the first that is missing or has another shape.
void check_layer_list_tensors(const ModelFile& file, const LayerListDesign& design);

}  // namespace qwen38
