// The BQ family (Qwen3.8): 4/5/6/8-bit weights from a .q38 file, Gated DeltaNet + gated full attention layers, norms
// folded into the GEMM epilogues. This file holds its activations and the kernel sequence of one step.
#include <algorithm>

#include "step_model.h"

namespace qwen38 {

namespace {

constexpr int kMaxSplits = 64;
// From this run length on, a step's GDN layers use the chunked recurrence: a 64-token chunk costs about as much as
// a dozen sequential token updates.
constexpr int kGdnChunkedMinRun = 16;

class BqModel final : public StepModel {
 public:
  BqModel(const ModelFile& f, const RunnerOptions& o) : file(f), cfg(f.config()), embedding_(o.embedding) {
    QWEN38_CHECK(o.compute == ComputeDtype::BF16, cfg.architecture, " models run in bfloat16 only");
    for (int i = 0; i < cfg.num_layers; ++i) {
      const std::string name = std::to_string(i) + (cfg.is_attention[size_t(i)] ? ".attn.qkvg" : ".gdn.qkvz");
      proj_ld = std::max(proj_ld, int(file.tensor(name).shape[0]));
    }
  }

  size_t weight_bytes() const override { return ModelWeights::required_device_bytes(file, embedding_); }
  size_t host_weight_bytes() const override {
    return embedding_ == EmbeddingPlacement::Host ? size_t(file.tensor("embed").bytes) : 0;
  }
  kernels::KvDtype resolve_kv_dtype(kernels::KvDtype d) const override {
    QWEN38_CHECK(d != kernels::KvDtype::F32, cfg.architecture, ": the KV cache is int8 or bf16");
    return d == kernels::KvDtype::Auto ? kernels::KvDtype::Int8 : d;
  }
  size_t kv_page_bytes(kernels::KvDtype d) const override { return KvCache::page_bytes_all_layers(cfg, d); }
  size_t state_bytes_per_slot() const override { return GdnStatePool::bytes_per_slot(cfg); }
  void load_weights() override { weights_ = std::make_unique<ModelWeights>(file, embedding_); }
  std::unique_ptr<KvCache> make_kv(kernels::KvDtype d, int pages, int slots, int max_pages) const override {
    return std::make_unique<KvCache>(cfg, d, pages, slots, max_pages);
  }
  void make_state(int slots) override { state_ = std::make_unique<GdnStatePool>(cfg, slots); }
  void reset_slot(int slot, cudaStream_t s) override { state_->reset(slot, s); }
  void carve(Workspace& w, const StepContext& ctx) override;
  void forward(const StepContext& ctx, const StepBatch& b) override;
  void head(const StepContext& ctx, const HeadRows& rows, float* logits) override;
  const ModelWeights* bq_weights() const override { return weights_.get(); }
  const kernels::GemmWorkspace* gemm_workspace() const override { return &gemm_ws; }

 private:
  const ModelFile& file;
  ModelConfig cfg;
  EmbeddingPlacement embedding_;
  std::unique_ptr<ModelWeights> weights_;
  std::unique_ptr<GdnStatePool> state_;
  // side branch of the step: the a/b gate projection of a GDN layer needs only the layer's input, so it runs beside
  // the layer's (much larger) in-projection GEMM; fork / join events make it a parallel branch of the captured graph
  Event fork_ev, join_ev;
  int proj_ld = 0;

  // activations
  float* residual = nullptr;
  __nv_bfloat16* xbf = nullptr;
  float* partials = nullptr;
  __nv_bfloat16* proj = nullptr;
  float* ab = nullptr;
  float* qkv = nullptr;
  __nv_bfloat16* mixer = nullptr;
  __nv_bfloat16* act = nullptr;
  __half* q16 = nullptr;
  float* split = nullptr;
  __nv_bfloat16* lm_x = nullptr;   // gathered rows for the LM head of ragged prefill steps
  float* lm_partials = nullptr;
  kernels::GemmWorkspace gemm_ws;
  float* gdn_scratch = nullptr;    // chunked GDN recurrence (prefill): per-chunk U0 / W / P
  size_t gdn_scratch_floats = 0;
};

void BqModel::carve(Workspace& w, const StepContext& ctx) {
  const size_t T = size_t(ctx.max_tokens), R = size_t(ctx.max_rows), H = size_t(cfg.hidden_size);
  const size_t mixer_w = size_t(std::max(cfg.q_dim(), cfg.gdn_value_dim()));
  const size_t nv2 = 2 * size_t(std::max(1, cfg.linear_num_value_heads));
  const size_t gemm_partials = size_t(2) * size_t(ctx.num_sms) * 128 * 512;  // stream-K partial tiles of a 512-token pass
  gdn_scratch_floats = cfg.linear_num_value_heads > 0 && ctx.max_tokens >= kGdnChunkedMinRun
                           ? kernels::gdn_chunk_scratch_floats(ctx.max_tokens, ctx.max_rows, cfg.linear_num_value_heads)
                           : 0;
  residual = w.take<float>(T * H);
  xbf = w.take<__nv_bfloat16>(T * H);
  partials = w.take<float>(T * size_t(cfg.norm_blocks()));
  proj = w.take<__nv_bfloat16>(T * size_t(proj_ld));
  ab = w.take<float>(T * nv2);
  qkv = w.take<float>(T * size_t(std::max(128, cfg.gdn_conv_dim())));
  mixer = w.take<__nv_bfloat16>(T * mixer_w);
  act = w.take<__nv_bfloat16>(T * size_t(cfg.intermediate_size));
  q16 = w.take<__half>(T * size_t(std::max(256, cfg.q_dim())));
  split = w.take<float>(R * size_t(std::max(1, cfg.num_attention_heads)) * kMaxSplits * (kernels::kHeadDim + 2));
  lm_x = w.take<__nv_bfloat16>(R * H);
  lm_partials = w.take<float>(R * size_t(cfg.norm_blocks()));
  gemm_ws.partials = w.take<float>(gemm_partials);
  gemm_ws.partial_floats = gemm_partials;
  gemm_ws.counters = w.take<int>(65536);
  gemm_ws.num_counters = 65536;
  gdn_scratch = w.take<float>(gdn_scratch_floats);
}

// The kernel sequence of one step over b.m tokens (reference src/model_runner.cpp:292-410).
void BqModel::forward(const StepContext& ctx, const StepBatch& b) {
  cudaStream_t s = ctx.stream;
  const int m = b.m;
  const bool decode = b.decode, mixed = b.mixed;
  const kernels::BatchDesc &batch = b.all, &chunk_part = b.chunk_part, &single_part = b.single_part;
  const int H = cfg.hidden_size;
  const float eps = cfg.rms_norm_eps;
  const kernels::KvCacheDesc kvd = ctx.kv->desc();
  const kernels::GdnStateDesc sd = state_->desc();
  kernels::GdnDims gd;
  gd.num_k_heads = cfg.linear_num_key_heads;
  gd.num_v_heads = cfg.linear_num_value_heads;
  gd.conv_dim = cfg.gdn_conv_dim();
  gd.ld_proj = proj_ld;

  kernels::embed(weights_->embedding(), b.tokens, m, H, residual, xbf, partials, s);
  ctx.mark("embed");

  kernels::GemmEpilogue into_residual;
  into_residual.kind = kernels::Epilogue::Residual;
  into_residual.residual = residual;
  into_residual.xbf = xbf;
  into_residual.partials_out = partials;

  int attn_i = 0, gdn_i = 0;
  for (const LayerWeights& W : weights_->layers()) {
    kernels::GemmEpilogue in;
    in.kind = kernels::Epilogue::StoreBF16;
    in.out = proj;
    in.ldo = proj_ld;
    in.n_store = W.in_proj.rows;
    in.partials_in = partials;
    in.hidden = H;
    in.eps = eps;
    const bool side_ab = !W.attention && !ctx.profiling;  // the per-op profile keeps everything on one stream
    if (side_ab) {
      fork_ev.record(s);
      QWEN38_CUDA(cudaStreamWaitEvent(ctx.side, fork_ev.get(), 0));
      kernels::gdn_ab(xbf, m, H, W.ab, W.ab_rows, partials, eps, ab, ctx.side);
      join_ev.record(ctx.side);
    }
    kernels::qgemm(xbf, m, W.in_proj, in, gemm_ws, s);
    ctx.mark(W.attention ? "gemm.attn_qkvg" : "gemm.gdn_qkvz");
    if (W.attention) {
      kernels::QkNormRopeParams qp;
      qp.proj = proj;
      qp.ld_proj = proj_ld;
      qp.q_norm = W.q_norm;
      qp.k_norm = W.k_norm;
      qp.eps = eps;
      qp.rope_theta = float(cfg.rope_theta);
      qp.num_q_heads = cfg.num_attention_heads;
      qp.num_kv_heads = cfg.num_key_value_heads;
      qp.q_out = q16;
      qp.attn_layer = attn_i;
      kernels::qk_norm_rope_append(qp, batch, kvd, s);
      ctx.mark("attn.qk_norm_rope_kv");
      kernels::AttentionParams ap;
      ap.q = q16;
      ap.gate = proj + cfg.q_dim();
      ap.ld_gate = proj_ld;
      ap.out = mixer;
      ap.num_q_heads = cfg.num_attention_heads;
      ap.num_kv_heads = cfg.num_key_value_heads;
      ap.attn_layer = attn_i;
      ap.split_scratch = split;
      ap.max_splits = kMaxSplits;
      if (decode) {
        kernels::attention_decode(ap, batch, kvd, s);
      } else if (mixed) {
        // chunk rows through the query-tiled kernel (no key split: the scratch serves the single-token rows), the
        // single-token rows through split-KV flash decoding
        kernels::attention_decode(ap, single_part, kvd, s);
        ap.split_scratch = nullptr;
        kernels::attention_prefill(ap, chunk_part, kvd, s);
      } else {  // the scratch of ctx.max_rows x kMaxSplits states seen as one row per prompt token of this step
        ap.max_splits = std::min(kMaxSplits, int(size_t(ctx.max_rows) * kMaxSplits / size_t(std::max(1, m))));
        ap.scratch_rows = ap.max_splits > 1 ? m : 0;
        kernels::attention_prefill(ap, batch, kvd, s);
      }
      ctx.mark(decode ? "attn.decode" : "attn.prefill");
      ++attn_i;
    } else {
      if (side_ab) QWEN38_CUDA(cudaStreamWaitEvent(s, join_ev.get(), 0));
      else kernels::gdn_ab(xbf, m, H, W.ab, W.ab_rows, partials, eps, ab, s);
      ctx.mark("gdn.ab");
      kernels::GdnConvParams cp;
      cp.proj = proj;
      cp.conv_w = W.conv;
      cp.qkv = qkv;
      cp.gdn_layer = gdn_i;
      kernels::gdn_conv(cp, gd, batch, sd, s);
      ctx.mark("gdn.conv");
      kernels::GdnRecurrenceParams rp;
      rp.qkv = qkv;
      rp.ab = ab;
      rp.A = W.A;
      rp.dt_bias = W.dt_bias;
      rp.z = proj + cfg.gdn_conv_dim();
      rp.ld_z = proj_ld;
      rp.norm_w = W.gdn_norm;
      rp.eps = eps;
      rp.out = mixer;
      rp.gdn_layer = gdn_i;
      // runs of prefill length take the chunked form (token-parallel preparation + per-chunk state scan)
      if (gdn_scratch && chunk_part.max_tokens_per_seq >= kGdnChunkedMinRun)
        kernels::gdn_recurrence_chunked(rp, gd, chunk_part, sd, gdn_scratch, gdn_scratch_floats, s);
      else
        kernels::gdn_recurrence(rp, gd, chunk_part, sd, s);
      if (mixed) kernels::gdn_recurrence(rp, gd, single_part, sd, s);  // the state-streaming decode kernel
      ctx.mark("gdn.recurrence");
      ++gdn_i;
    }
    kernels::qgemm(mixer, m, W.out_proj, into_residual, gemm_ws, s);
    ctx.mark(W.attention ? "gemm.attn_o" : "gemm.gdn_out");

    kernels::GemmEpilogue mlp;
    mlp.kind = kernels::Epilogue::SwiGLU;
    mlp.out = act;
    mlp.ldo = cfg.intermediate_size;
    mlp.partials_in = partials;
    mlp.hidden = H;
    mlp.eps = eps;
    kernels::qgemm(xbf, m, W.gate_up, mlp, gemm_ws, s);
    ctx.mark("gemm.mlp_gate_up");
    kernels::qgemm(act, m, W.down, into_residual, gemm_ws, s);
    ctx.mark("gemm.mlp_down");
  }
}

void BqModel::head(const StepContext& ctx, const HeadRows& rows, float* logits) {
  const __nv_bfloat16* x = xbf + size_t(rows.first) * size_t(cfg.hidden_size);
  const float* part = partials + size_t(rows.first) * size_t(cfg.norm_blocks());
  if (rows.rows) {
    kernels::gather_rows(xbf, partials, rows.rows, rows.count, cfg.hidden_size, lm_x, lm_partials, ctx.stream);
    x = lm_x;
    part = lm_partials;
  }
  kernels::GemmEpilogue head;
  head.kind = kernels::Epilogue::StoreF32;
  head.out = logits;
  head.ldo = cfg.vocab_size;
  head.partials_in = part;
  head.hidden = cfg.hidden_size;
  head.eps = cfg.rms_norm_eps;
  kernels::qgemm(x, rows.count, weights_->lm_head(), head, gemm_ws, ctx.stream);
  ctx.mark("gemm.lm_head");
}

const ArchitectureRegistration registration{{"Qwen3.8", nullptr, nullptr,
                                             [](const ModelFile& f, const RunnerOptions& o) -> std::unique_ptr<StepModel> {
                                               return std::make_unique<BqModel>(f, o);
                                             }}};

}  // namespace

}  // namespace qwen38
