// Shared between the translation units of the mixed-head attention (mixed_attention.cu, mixed_attention_mma.cu).
#pragma once

#include "host_util.h"

namespace q38 {

// Tensor-core forms (bf16 cache). `can_*` say whether the shape fits; otherwise the general kernels serve the call.
bool mixed_prefill_mma_fits(const q38_mixed_attention_params& p, const q38_kv_layer_desc& kv);
int mixed_prefill_mma(const q38_mixed_attention_params& p, const q38_batch_desc& b, const q38_kv_layer_desc& kv, cudaStream_t s);
bool mixed_decode_mma_fits(const q38_mixed_attention_params& p, const q38_kv_layer_desc& kv);
int mixed_decode_mma(const q38_mixed_attention_params& p, const q38_batch_desc& b, const q38_kv_layer_desc& kv, cudaStream_t s);

}  // namespace q38
