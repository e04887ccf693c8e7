// What a model architecture provides to the step executor. ModelRunner owns everything that is the same for every
// architecture - slots and pages, the ragged step metadata, CUDA graphs, sampling, scoring, error status - and calls
// a StepModel for its weights, its per-sequence state and the kernel sequence of one step. Architectures register
// themselves by the name their model files carry (Architecture below).
#pragma once

#include "json_min.h"
#include "qwen38/api.h"

namespace qwen38 {

inline size_t up256(size_t x) { return (x + 255) / 256 * 256; }

// Activation memory in two passes over the same code: without an arena the requests are only added up, with one they
// are handed out.
struct Workspace {
  DeviceArena* arena = nullptr;
  size_t bytes = 0;
  template <typename T>
  T* take(size_t count) {
    bytes += up256(count * sizeof(T));
    return arena && count ? arena->allocate_array<T>(count) : nullptr;
  }
};

// The executor's services a model uses while it builds or runs a step.
struct StepContext {
  cudaStream_t stream = nullptr;
  cudaStream_t side = nullptr;  // parallel branch of the step (fork / join by events)
  int num_sms = 0;
  int max_tokens = 0, max_rows = 0;
  KvCache* kv = nullptr;
  bool profiling = false;
  std::function<void(const char*)> mark;  // per-op profile: the op of this name has just been enqueued
};

// One step: the tokens of all its sequences as one ragged batch. In a mixed step the sequences that bring several
// tokens (chunk_part) come before those that bring one (single_part); otherwise both parts are the whole batch.
struct StepBatch {
  const int32_t* tokens = nullptr;  // [m] device
  int m = 0;
  bool decode = false, mixed = false;
  kernels::BatchDesc all, chunk_part, single_part;
  // prefill steps: the longest context of a sequence of chunk_part, and the sum of all of them in whole pages (tokens)
  int chunk_longest_context = 0;
  int64_t chunk_packed_rows = 0;
};

// Token rows of the last forward() whose logits are wanted: `count` rows from `first`, or, with `rows` (device), those.
struct HeadRows {
  const int* rows = nullptr;
  int first = 0, count = 0;
};

class StepModel {
 public:
  virtual ~StepModel() = default;
  // memory plan
  virtual size_t weight_bytes() const = 0;
  virtual size_t host_weight_bytes() const { return 0; }
  virtual kernels::KvDtype resolve_kv_dtype(kernels::KvDtype requested) const = 0;
  virtual size_t kv_page_bytes(kernels::KvDtype dtype) const = 0;
  virtual size_t state_bytes_per_slot() const = 0;
  virtual void carve(Workspace& ws, const StepContext& ctx) = 0;
  // allocation
  virtual void load_weights() = 0;
  virtual std::unique_ptr<KvCache> make_kv(kernels::KvDtype dtype, int pages, int slots, int max_pages_per_seq) const = 0;
  virtual void make_state(int slots) = 0;
  // once the workspace exists (and has been zeroed), before the first step
  virtual void prepare(const StepContext&) {}
  // the step
  virtual void reset_slot(int slot, cudaStream_t stream) = 0;
  virtual void forward(const StepContext& ctx, const StepBatch& batch) = 0;
  virtual void head(const StepContext& ctx, const HeadRows& rows, float* logits) = 0;
  // BQ models only
  virtual const ModelWeights* bq_weights() const { return nullptr; }
  virtual const kernels::GemmWorkspace* gemm_workspace() const { return nullptr; }
};

// A registered architecture. `read_config` turns a model folder's config.json into the configuration (null for
// architectures that only exist as .q38 files, whose header the file reader knows).
struct Architecture {
  const char* name;
  ModelConfig (*read_config)(const jsonmin::Value& config);
  void (*check_tensors)(const ModelFile& file);
  std::unique_ptr<StepModel> (*make)(const ModelFile& file, const RunnerOptions& options);
};
void register_architecture(const Architecture& a);
const Architecture& find_architecture(const std::string& name);  // throws Error with the known names
std::vector<std::string> architecture_names();
struct ArchitectureRegistration {
  explicit ArchitectureRegistration(const Architecture& a) { register_architecture(a); }
};

}  // namespace qwen38
