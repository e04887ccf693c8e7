/* q38_kernels.h — C ABI of the B200 (sm_100a) kernels of the ragged continuous-batching step.
 *
 * This is the drop-in boundary: every entry point replaces one launcher of the reference's internal
 * kernel API `src/kernels/kernels.h` (namespace qwen38::kernels). Signatures use plain pointers,
 * sizes and POD structs only (no C++ or torch types), so the library can be bound from C, C++, or any
 * FFI. The contract of the reference launchers is kept (src/kernels/kernels.h:3-6):
 *   - activations are row-major, M = number of tokens of the step;
 *   - every pointer is a device pointer unless stated otherwise (the embedding table may be mapped
 *     pinned host memory);
 *   - every launcher is asynchronous on `stream` (a cudaStream_t passed as void*; NULL = the legacy
 *     default stream), allocates nothing, never synchronises the host and may be captured into a CUDA
 *     graph: all data-dependent sizes are read from device memory, only `num_seqs`, `num_tokens` and
 *     `max_tokens_per_seq` are host values fixed per captured graph.
 * Errors: launchers validate arguments on the host and return Q38_OK or a negative code; the message
 * is available from q38_last_error(). Kernels never trap or assert; bounded device-side waits report
 * through q38_device_error().
 */
#ifndef Q38_KERNELS_H_
#define Q38_KERNELS_H_

#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

#define Q38_OK 0
#define Q38_ERR_INVALID (-1) /* argument validation failed (reference: QWEN38_CHECK -> qwen38::Error) */
#define Q38_ERR_CUDA (-2)    /* a CUDA runtime / driver call made by the launcher failed */

#define Q38_PAGE_TOKENS 64 /* src/kernels/kernels.h:38 kPageTokens */
#define Q38_HEAD_DIM 256   /* src/kernels/kernels.h:39 kHeadDim */

typedef uint16_t q38_bf16; /* raw bfloat16 bits */
typedef uint16_t q38_f16;  /* raw IEEE half bits */

/* Ragged batch of one step. Replaces kernels::BatchDesc (src/kernels/kernels.h:22-31). */
typedef struct q38_batch_desc {
  int num_seqs;           /* B (host value) */
  int num_tokens;         /* M (host value) */
  int max_tokens_per_seq; /* upper bound of a sequence's run length in this step (host value) */
  const int* seq_start;   /* [B + 1] */
  const int* seq_slot;    /* [B] state slot = block-table row */
  const int* seq_pos0;    /* [B] position of the sequence's first token of this step */
  const int* tok_pos;     /* [M] absolute position of every token */
  const int* tok_seq;     /* [M] sequence index of every token */
} q38_batch_desc;

/* Paged KV cache. Replaces kernels::KvCacheDesc (src/kernels/kernels.h:36-70); the byte layout of a
 * (layer, page) block is the reference's: K [kv_head][64][256], V same, then for int8 the fp16 scales
 * K [kv_head][64][4], V same. */
#define Q38_KV_INT8 0
#define Q38_KV_BF16 1
#define Q38_KV_F32 2 /* q38_kv_layer_desc only */
typedef struct q38_kv_cache_desc {
  uint8_t* pool;
  int dtype; /* Q38_KV_INT8 | Q38_KV_BF16 */
  int kv_heads;
  int num_pages;
  size_t page_bytes;
  size_t layer_stride;
  const int* block_table; /* [slots][max_pages_per_seq] */
  int max_pages_per_seq;
} q38_kv_cache_desc;
size_t q38_kv_page_bytes(int dtype, int kv_heads); /* KvCacheDesc::page_bytes_for, kernels.h:66-69 */

/* BQ weight (reference docs/FORMAT.md section 2). Replaces kernels::BQWeight (kernels.h:82-90). */
typedef struct q38_bq_weight {
  const uint8_t* lo;
  const uint8_t* hi;      /* NULL for 4-bit */
  const q38_bf16* scales;
  int bits;               /* 4, 5, 6, 8 */
  int n;                  /* padded rows, multiple of 128 */
  int k;                  /* multiple of 64 */
  int rows;               /* logical rows */
} q38_bq_weight;

/* GEMM epilogues. Replaces kernels::Epilogue / GemmEpilogue / GemmWorkspace (kernels.h:75-111). */
#define Q38_EPI_STORE_BF16 0 /* out = bf16(C * rs) */
#define Q38_EPI_SWIGLU 1     /* out[i] = bf16(silu(C[2i] * rs) * C[2i+1] * rs) */
#define Q38_EPI_RESIDUAL 2   /* residual += C; xbf = bf16(residual); partials_out = sum of squares / 128 cols */
#define Q38_EPI_STORE_F32 3  /* out = C * rs */
/* Tensor parallelism, row-parallel projections of up to 16 tokens: C is this rank's partial product. The GEMM kernel
 * itself stores each finished 128-column tile into every rank's receive buffer (plain peer stores over NVLink), raises
 * a per-tile flag there, waits - bounded - for the other ranks' flags in its own memory, sums the pieces in rank order
 * (every rank gets the same bits) and then runs the Residual epilogue on the sum. No counterpart in the reference
 * (single GPU); replaces the all-reduce a host would otherwise place between q38_qgemm and q38_residual_update. */
#define Q38_EPI_ALLREDUCE_RESIDUAL 4
#define Q38_MAX_PEERS 8
#define Q38_ALLREDUCE_ROWS 16
typedef struct q38_peer_allreduce {
  int world, rank;
  /* rank r's receive buffer as mapped into this process, [2][world][Q38_ALLREDUCE_ROWS][n] floats (two buffers used in
   * turn), and its flags, [n / 128][world] words; entry `rank` is this rank's own memory. All zero before first use. */
  float* recv[Q38_MAX_PEERS];
  unsigned int* flags[Q38_MAX_PEERS];
  unsigned int* seq;       /* this rank's call counters, [n / 128] words, zero before first use */
  unsigned int poll_limit; /* polls of a flag before the wait gives up and sets q38_device_error(); 0 = 2^22 */
} q38_peer_allreduce;
typedef struct q38_gemm_epilogue {
  int kind;
  void* out;
  int ldo;
  int n_store;
  float* residual;
  q38_bf16* xbf;
  float* partials_out;
  const float* partials_in; /* rs = rsqrt(sum(partials_in[row]) / hidden + eps); NULL = 1 */
  int hidden;
  float eps;
  const q38_peer_allreduce* allreduce; /* Q38_EPI_ALLREDUCE_RESIDUAL only; NULL otherwise */
} q38_gemm_epilogue;

typedef struct q38_gemm_workspace {
  float* partials;       /* stream-K partial tiles */
  size_t partial_floats;
  int* counters;         /* per-tile arrival counters: zeroed once by the caller, self-resetting */
  int num_counters;
} q38_gemm_workspace;

/* kernels.h:113-125 */
#define Q38_GEMM_CONFIG_AUTO (-1)
int q38_qgemm_num_configs(void);
const char* q38_qgemm_config_name(int config);
int q38_qgemm_config_tile_m(int config);
/* The configuration q38_qgemm picks for Q38_GEMM_CONFIG_AUTO: the installed tuning lookup's answer if it has one,
 * else the built-in rule (pure host logic, no device access; no counterpart in the reference, whose launcher keeps
 * the choice to itself - tools use it to report what "auto" meant). */
int q38_qgemm_auto_config(int bits, int n, int k, int m);
/* C[M][N] = A[M][K] * W^T; A bf16 row-major with leading dimension K. (kernels::qgemm, kernels.h:120-121) */
int q38_qgemm(const q38_bf16* a, int m, const q38_bq_weight* w, const q38_gemm_epilogue* ep,
              const q38_gemm_workspace* ws, void* stream, int config);
/* The same GEMM for callers that cannot allocate device memory (no counterpart in the reference, whose launcher
 * always receives a caller-owned GemmWorkspace). The stream-K workspace is a fixed array inside the library
 * (about 3.2 MB of device memory per GPU that loads it). Limits: 1 <= m <= 16, n <= 524288, at most 192 SMs;
 * anything larger is rejected with Q38_ERR_INVALID. The first call on a device looks the array's address up
 * (cudaGetSymbolAddress) and should therefore be made before any stream capture starts. Every call on a device
 * uses the same array: calls that may overlap on the GPU must be serialised by the caller. Allocates nothing. */
int q38_qgemm_static(const q38_bf16* a, int m, const q38_bq_weight* w, const q38_gemm_epilogue* ep, void* stream);
typedef int (*q38_gemm_tuning_lookup)(int bits, int n, int k, int m);
void q38_set_qgemm_tuning(q38_gemm_tuning_lookup lookup); /* kernels::set_qgemm_tuning, kernels.h:124-125 */

/* Dequantised weights W[n][k] as bf16 (row-major, padded rows included): the values the GEMM feeds to
 * the tensor cores. Test / inspection helper of the in-register decoder (the reference checks the same
 * logic on the host, tests/host/test_bq_layout.cpp). */
int q38_bq_dequant(const q38_bq_weight* w, q38_bf16* out, void* stream);

/* kernels::embed, kernels.h:131-134 */
int q38_embed(const q38_bf16* table, const int32_t* tokens, int m, int hidden, float* residual, q38_bf16* xbf,
              float* partials, void* stream);

/* The Residual GEMM epilogue as an op of its own: residual += delta, xbf = bf16(residual), partials[m][col / 128] =
 * sum of squares. For tensor-parallel runs, where the row-parallel projections store fp32 partial products
 * (Q38_EPI_STORE_F32) that are summed over the ranks first. No counterpart in the reference (single GPU). */
int q38_residual_update(const float* delta, int m, int hidden, float* residual, q38_bf16* xbf, float* partials,
                        void* stream);

/* Device memory that other processes of the node can map (buffers and flags of Q38_EPI_ALLREDUCE_RESIDUAL): allocation
 * (zero-filled), the 64-byte handle a peer process opens, opening and closing a peer's handle. The handles travel
 * through whatever the host uses between its ranks. One process per GPU; peer access is enabled on opening. */
int q38_peer_alloc(size_t bytes, void** ptr);
int q38_peer_free(void* ptr);
int q38_peer_export(void* ptr, unsigned char handle[64]);
int q38_peer_open(const unsigned char handle[64], void** ptr);
int q38_peer_close(void* ptr);

/* Packs rows rows[0..n) of the step's LM-head inputs (bf16 hidden rows x [M][hidden] and their norm partial sums
 * [M][hidden / 128]) into rows 0..n-1 of x_out / partials_out: the last-token rows of the sequences that sample in a
 * ragged step. Replaces the per-row device copies of the reference's prefill path (src/model_runner.cpp:471-489 reads
 * one row; a ragged step has up to one per sequence). `rows` is a device array. */
int q38_gather_rows(const q38_bf16* x, const float* partials, const int* rows, int n, int hidden, q38_bf16* x_out,
                    float* partials_out, void* stream);

/* kernels::QkNormRopeParams + qk_norm_rope_append, kernels.h:140-155 */
typedef struct q38_qk_norm_rope_params {
  const q38_bf16* proj; /* [M][ld_proj]: [q | gate | k | v] */
  int ld_proj;
  const float* q_norm;  /* [256], already 1 + w */
  const float* k_norm;
  float eps;
  float rope_theta;
  int num_q_heads;
  int num_kv_heads;
  q38_f16* q_out;       /* [M][nq][256] */
  int attn_layer;
} q38_qk_norm_rope_params;
int q38_qk_norm_rope_append(const q38_qk_norm_rope_params* p, const q38_batch_desc* batch,
                            const q38_kv_cache_desc* kv, void* stream);

/* kernels::AttentionParams, attention_decode_splits, attention_decode, attention_prefill, kernels.h:157-179 */
typedef struct q38_attention_params {
  const q38_f16* q;      /* [M][nq][256] */
  const q38_bf16* gate;  /* proj + nq*256, row stride ld_gate */
  int ld_gate;
  q38_bf16* out;         /* [M][nq*256] */
  int num_q_heads;
  int num_kv_heads;
  int attn_layer;
  float* split_scratch;  /* [B][nq][max_splits][256 + 2] floats */
  int max_splits;
  /* Extension (not in the reference's struct): rows B the scratch was sized for. Decode needs one row per sequence
   * and ignores the field. Prefill cuts the keys of its query tiles over several CTAs only when there are few tiles
   * for the GPU (one long request, a tensor-parallel rank with one kv head) and only if the scratch holds one row
   * per prompt token of the step: scratch_rows >= num_tokens. 0 = sized for the decode batch only (never split). */
  int scratch_rows;
} q38_attention_params;
int q38_attention_decode_splits(int batch_seqs, int kv_heads, int num_sms, int max_splits);
int q38_attention_decode(const q38_attention_params* p, const q38_batch_desc* batch, const q38_kv_cache_desc* kv,
                         void* stream);
int q38_attention_prefill(const q38_attention_params* p, const q38_batch_desc* batch, const q38_kv_cache_desc* kv,
                          void* stream);

/* kernels::GdnDims / GdnStateDesc, kernels.h:184-195 */
typedef struct q38_gdn_dims {
  int num_k_heads;
  int num_v_heads;
  int conv_dim; /* 2 * nk * 128 + nv * 128 */
  int ld_proj;
} q38_gdn_dims;
typedef struct q38_gdn_state_desc {
  float* recurrent;  /* [slots][gdn_layers][nv][128 dv][128 dk] */
  q38_bf16* conv;    /* [slots][gdn_layers][3][conv_dim] */
  int num_gdn_layers;
} q38_gdn_state_desc;

/* kernels::gdn_ab, kernels.h:197-199 */
int q38_gdn_ab(const q38_bf16* xbf, int m, int hidden, const q38_bf16* w_ab, int rows, const float* partials_in,
               float eps, float* ab_out, void* stream);

/* kernels::GdnConvParams + gdn_conv, kernels.h:201-210 */
typedef struct q38_gdn_conv_params {
  const q38_bf16* proj;
  const float* conv_w; /* [conv_dim][4] */
  float* qkv;          /* [M][conv_dim] */
  int gdn_layer;
} q38_gdn_conv_params;
int q38_gdn_conv(const q38_gdn_conv_params* p, const q38_gdn_dims* d, const q38_batch_desc* batch,
                 const q38_gdn_state_desc* st, void* stream);

/* kernels::GdnRecurrenceParams + gdn_recurrence, kernels.h:212-228 */
typedef struct q38_gdn_recurrence_params {
  const float* qkv;
  const float* ab;
  const float* A;
  const float* dt_bias;
  const q38_bf16* z;
  int ld_z;
  const float* norm_w;
  float eps;
  q38_bf16* out;
  int gdn_layer;
} q38_gdn_recurrence_params;
int q38_gdn_recurrence(const q38_gdn_recurrence_params* p, const q38_gdn_dims* d, const q38_batch_desc* batch,
                       const q38_gdn_state_desc* st, void* stream);

/* The same operation in the chunked (64-token WY) form for prefill-sized runs: token-parallel preparation plus a
 * per-chunk state scan instead of a token-by-token loop; results agree with q38_gdn_recurrence to fp32 rounding.
 * Any run lengths are accepted (short runs are padded to a chunk, so q38_gdn_recurrence is the better choice when
 * batch->max_tokens_per_seq is small). `scratch` holds q38_gdn_chunk_scratch_floats(num_tokens, num_seqs,
 * num_v_heads) floats, 16-byte aligned, and may be reused by the next call on the same stream.
 * No counterpart in the reference, whose gdn_recurrence (kernels.h:212-228) is token-sequential. */
size_t q38_gdn_chunk_scratch_floats(int max_tokens, int max_seqs, int num_v_heads);
int q38_gdn_recurrence_chunked(const q38_gdn_recurrence_params* p, const q38_gdn_dims* d,
                               const q38_batch_desc* batch, const q38_gdn_state_desc* st, float* scratch,
                               size_t scratch_floats, void* stream);
/* Which form of the chunk scan q38_gdn_recurrence_chunked launches: 1 (default) = the four per-chunk products on the
 * tensor cores (mma.sync TF32 with every factor split into two TF32 numbers, three MMAs per product: fp32-like
 * accuracy, fp32 sums), 0 = all fp32 on the CUDA cores. Process-wide; applies to launches made after the call. No
 * counterpart in the reference (its recurrence is token-sequential). */
void q38_gdn_set_chunk_scan_tensor_cores(int on);

/* kernels::SamplingParamsDev / SamplingArgs / sample / target_logprobs, kernels.h:233-260 */
typedef struct q38_sampling_params_dev {
  float temperature;
  int top_k;
  float top_p;
  float min_p;
  float presence_penalty;
  float repetition_penalty;
  uint64_t seed;
} q38_sampling_params_dev;
typedef struct q38_sampling_args {
  float* logits;
  int ld;
  int vocab;
  const q38_sampling_params_dev* params;
  const int* row_slot;
  int32_t* history;
  int* history_len;
  int history_cap;
  const int* step;
  int32_t* tokens_out;
  float* logprob_out;
} q38_sampling_args;
int q38_sample(const q38_sampling_args* a, int batch, void* stream);
int q38_target_logprobs(const float* logits, int ld, int vocab, const int32_t* targets, int rows, float* out,
                        void* stream);

/* Ragged-batch packing on the GPU. Replaces the host loops that fill the step metadata
 * (src/model_runner.cpp:458-469 for prefill, :534-560 for decode): expands per-sequence
 * (slot, pos0, count) rows into seq_start / tok_pos / tok_seq. Inputs are device arrays of num_seqs
 * entries; outputs are the arrays a q38_batch_desc points at. num_tokens must equal sum(count). */
int q38_pack_ragged(const int* seq_count, const int* seq_pos0, int num_seqs, int num_tokens, int* seq_start,
                    int* tok_pos, int* tok_seq, void* stream);

/* ---------------------------------------------------------------------------------------------------------------
 * Layer-list architectures with dense (bf16) weights: decoders whose configuration lists a mixer and an optional gated
 * feed-forward per layer. No counterpart in the reference. Activations are bf16 or fp32 (`act`); with Q38_ACT_F32 every
 * product is computed in 32-bit. Rows of activation matrices start every `ld` elements; the elements between a row's
 * length and `ld` must be finite (they meet zero weights).
 * ------------------------------------------------------------------------------------------------------------- */
#define Q38_ACT_BF16 0
#define Q38_ACT_F32 1

/* One attention layer's pages: page p at pages + p * page_bytes, first K [kv_head][64 tokens][k_dim], then V transposed,
 * [kv_head][v_dim][64 tokens]; k_dim is a multiple of 32, v_dim of 8 (heads are padded with zeros). */
typedef struct q38_kv_layer_desc {
  uint8_t* pages;
  int dtype; /* Q38_KV_BF16 | Q38_KV_F32, equal to the activations' precision */
  int kv_heads, k_dim, v_dim;
  int num_pages;
  size_t page_bytes;
  const int* block_table; /* [slots][max_pages_per_seq] */
  int max_pages_per_seq;
} q38_kv_layer_desc;

/* One recurrent layer's state: slot s at byte offset s * slot_bytes of both pointers. `state` is fp32 [width] (retention:
 * [heads][dim][vdim]); `conv` is a ring [taps][channels] in activation precision, the input of position p in row p % taps. Positions before the
 * sequence's start are zero and are never read, so a fresh sequence needs no clearing: at position 0 the recurrence
 * starts from zero by itself. */
typedef struct q38_recurrent_state_desc {
  uint8_t* state;
  uint8_t* conv;
  size_t slot_bytes;
} q38_recurrent_state_desc;

/* y[m][n] = x[m][k] W^T + bias. W bf16 [n][k], rows `ld` elements apart (a multiple of 64, zero beyond k), with zero
 * rows up to a multiple of 16. */
typedef struct q38_dense_weight {
  const q38_bf16* w;
  const float* bias; /* [n] or NULL */
  int n, k, ld;
} q38_dense_weight;
#define Q38_DENSE_STORE 0     /* out[m][n] in activation precision */
#define Q38_DENSE_STORE_F32 1 /* out[m][n] fp32 */
#define Q38_DENSE_GLU_GELU 2  /* rows of W alternate gate, up: out[m][n / 2] = gelu_tanh(gate) * up, activation precision */
#define Q38_DENSE_GLU_SILU 3  /* the same with silu */
#define Q38_DENSE_XIELU 4     /* out[m][n] = xielu(y), activation precision: alpha_p y^2 + y / 2 for y > 0,
                               * alpha_n (e^y - 1 - y) + y / 2 below */
#define Q38_DENSE_GATE_SIGMOID 5 /* out[m][n] = y * sigmoid(gate[m][n]), both in activation precision */
typedef struct q38_dense_epilogue {
  int kind;
  void* out;
  int ldo;
  float alpha_p, alpha_n; /* Q38_DENSE_XIELU */
  const void* gate;       /* Q38_DENSE_GATE_SIGMOID */
  int ld_gate;
} q38_dense_epilogue;
#define Q38_DENSE_AUTO (-1)
int q38_dense_gemm_num_configs(void);
const char* q38_dense_gemm_config_name(int config);
int q38_dense_gemm(const void* x, int ldx, int act, int m, const q38_dense_weight* w, const q38_dense_epilogue* ep,
                   const q38_gemm_workspace* ws, void* stream, int config);
/* Several products of one shape side by side: group g multiplies columns g * x_stride ... of x (k of them; x_stride a
 * multiple of 8 elements) with rows g * n ... of W and writes columns g * out_stride ... of out (and of the gate). */
typedef struct q38_dense_groups {
  int count, x_stride, out_stride;
} q38_dense_groups;
int q38_dense_gemm_grouped(const void* x, int ldx, int act, int m, const q38_dense_weight* w, const q38_dense_groups* groups,
                           const q38_dense_epilogue* ep, const q38_gemm_workspace* ws, void* stream, int config);

/* RMS norm with a gain per coordinate (gain_stride 1) or one gain for all (gain_stride 0); `out` in activation precision.
 * With groups > 1 (the stream kernels below) each of `groups` equal consecutive parts of the row has its own root mean
 * square; 0 or 1 = the whole row. */
typedef struct q38_norm {
  const float* gain;
  int gain_stride;
  float eps;
  int groups;
} q38_norm;
/* residual = table[token] (+ positions[position] if not NULL); out = norm(residual) */
int q38_embed_norm(const q38_bf16* table, const q38_bf16* positions, const int32_t* tokens, const int* tok_pos, int m,
                   int width, float* residual, const q38_norm* norm, void* out, int ld_out, int act, void* stream);
/* residual += post(y); out = next(residual) unless next is NULL. Post-norm, residual sum and the following sublayer's
 * pre-norm in one pass over the row. */
int q38_residual_norm(const float* y, int ldy, int m, int width, const q38_norm* post, float* residual,
                      const q38_norm* next, void* out, int ld_out, int act, void* stream);
/* out[i] = norm(residual[rows ? rows[i] : first + i]), i < n (rows is a device array) */
int q38_gather_norm(const float* residual, const int* rows, int first, int n, int width, const q38_norm* norm, void* out,
                    int ld_out, int act, void* stream);

/* Hyper-connections: the residual is `streams` rows per token, [m][streams][width] fp32. A sublayer reads
 * u = sum_s in[s] x_s through its pre-norm and its output y replaces all streams at once by
 * x_t = sum_s mix[s][t] x_s + mult * out[t] * y. One stream with in = out = mix = 1 is the ordinary residual sum. */
typedef struct q38_stream_update {
  const float* mix; /* [streams from][streams to] */
  const float* out; /* [streams] */
  float mult;
} q38_stream_update;
#define Q38_MAX_STREAMS 16
/* every stream = scale * table[token]; out = norm(sum_s in[s] x_s) */
int q38_stream_embed(const q38_bf16* table, const int32_t* tokens, int m, int width, float scale, int streams,
                     float* residual, const float* in, const q38_norm* norm, void* out, int ld_out, int act, void* stream);
/* The update of one sublayer, then the next one's u and pre-norm (unless next is NULL), in one pass over the row. */
int q38_stream_norm(const float* y, int ldy, int m, int width, int streams, const q38_stream_update* update, float* residual,
                    const float* in, const q38_norm* next, void* out, int ld_out, int act, void* stream);
/* out[i] = norm(sum of the streams of row rows ? rows[i] : first + i), i < n */
int q38_stream_gather(const float* residual, const int* rows, int first, int n, int width, int streams, const q38_norm* norm,
                      void* out, int ld_out, int act, void* stream);

/* Rotary positions on the leading rot_dims of every query and key head (dimension i turns with i + rot_dims / 2 by
 * position * inv_freq[i]), optional blending of the values with a first layer's, and the append to the cache.
 * proj rows: [q: heads x dim | k: kv_heads x dim | v: kv_heads x vdim]. */
typedef struct q38_rope_append_params {
  const void* proj;
  int ld_proj;
  int act;
  int heads, kv_heads, dim, vdim;
  int rot_dims;
  const double* inv_freq; /* [rot_dims / 2]: base^(-2 i / rot_dims) */
  void* q_out;            /* [M][heads][k_dim of the cache], zero beyond dim */
  void* v_first_out;      /* [M][kv_heads * vdim]: where to keep this layer's values, or NULL */
  const void* v_first_in; /* values to blend with, or NULL: v = (1 - *v_mix) v + *v_mix v_first */
  const float* v_mix;
} q38_rope_append_params;
int q38_rope_append(const q38_rope_append_params* p, const q38_batch_desc* batch, const q38_kv_layer_desc* kv, void* stream);

/* Causal attention over the cache whose heads' softmax weights are mixed before they meet the values:
 * w_h(i, j) = sum_g head_mix[h][g] softmax_g(i, j); head_mix NULL = no mixing. Query head h reads kv head
 * h / (heads / kv_heads). */
typedef struct q38_mixed_attention_params {
  const void* q; /* [M][heads][k_dim] */
  int act;
  int heads, vdim;
  float scale;
  const float* head_mix; /* [heads][heads] or NULL */
  void* out;             /* [M][ld_out]: heads x vdim */
  int ld_out;
  float* stats;          /* [max(1, stat_splits)][M][heads][2] */
  int stat_splits;       /* prefill: key ranges the normalisers may be computed in */
  float* scores;         /* decode: [num_pages][heads][64] (NULL: the decode call uses the prefill kernels) */
  float* partials;       /* decode: [num_seqs][max_splits][heads][v_dim of the cache + 2] */
  int max_splits;
} q38_mixed_attention_params;
int q38_mixed_attention_prefill(const q38_mixed_attention_params* p, const q38_batch_desc* batch,
                                const q38_kv_layer_desc* kv, void* stream);
int q38_mixed_attention_decode(const q38_mixed_attention_params* p, const q38_batch_desc* batch,
                               const q38_kv_layer_desc* kv, void* stream);

/* minGRU: proj rows [z | x | g], each `width`; z = sigmoid(z), candidate x + 1/2 (x >= 0) or sigmoid(x),
 * S = (1 - z) S + z candidate, out = S silu(g). */
typedef struct q38_mingru_params {
  const void* proj;
  int ld_proj;
  int act;
  int width;
  void* out;
  int ld_out;
} q38_mingru_params;
int q38_mingru(const q38_mingru_params* p, const q38_batch_desc* batch, const q38_recurrent_state_desc* st, void* stream);

/* Real-gated linear recurrent unit behind a causal convolution: proj rows [y | x], each `width`; u = conv(x) + conv_b;
 * r, i = sigmoid(block-diagonal products of u); log a = log_decay * r * softplus(lam); S = a S + sqrt(1 - a^2) i u;
 * out = S gelu_tanh(y). gate_w [blocks][2 (r, i)][block_ld][block_ld] bf16 with block_ld a multiple of 32, zero padded. */
typedef struct q38_rglru_params {
  const void* proj;
  int ld_proj;
  int act;
  int width, blocks, block_ld, taps;
  const float* conv_w; /* [taps][width], the last row meets the current token */
  const float* conv_b; /* [width] */
  const q38_bf16* gate_w;
  const float* gate_b; /* [2][width] */
  const float* lam;    /* [width] */
  float log_decay;     /* negative */
  float* scratch;      /* [2][num_tokens][width]; batches of one token per sequence do not use it */
  void* out;
  int ld_out;
} q38_rglru_params;
int q38_rglru(const q38_rglru_params* p, const q38_batch_desc* batch, const q38_recurrent_state_desc* st, void* stream);

/* Retention: linear attention with a fixed decay per head, S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t; q and k turn
 * on their leading rot_dims dimensions as in q38_rope_append and k is multiplied by k_scale after that; every head's o is
 * divided by its root mean square and multiplied by silu(g). proj rows: [q: heads x dim | k: heads x dim | v: heads x vdim
 * | g: heads x vdim]. Rotated q and k, decays, the state and o are fp32 (products of fp32 factors on the tensor cores run
 * on bf16 hi + lo terms). */
#define Q38_RETENTION_CHUNK 64
typedef struct q38_retention_params {
  const void* proj;
  int ld_proj;
  int act;
  int heads, dim, vdim;
  int rot_dims;
  const double* inv_freq;  /* [rot_dims / 2] */
  const float* decay_pow;  /* [heads][Q38_RETENTION_CHUNK + 1]: decay^i */
  float k_scale, eps;
  void* qk;                /* scratch, q38_retention_qk_bytes(num_tokens, ...); runs of one token per sequence use none */
  float* o;                /* scratch [M][heads * vdim]; likewise */
  void* out;
  int ld_out;
} q38_retention_params;
size_t q38_retention_qk_bytes(int tokens, int heads, int dim, int act);
int q38_retention(const q38_retention_params* p, const q38_batch_desc* batch, const q38_recurrent_state_desc* st, void* stream);

/* Latent attention: queries and keys meet in the latent space of the cache. The cache (kv_heads 1, v_dim 0) holds one
 * normalised latent c of k_dim numbers per token, which is key and value at once; the heads' key and value matrices are
 * applied to the queries before and to the outputs after (q38_dense_gemm_grouped).
 * Append: proj rows [query latent: q_rank | kv latent: kv_rank | ...], each divided by its root mean square and multiplied
 * by its gain; the query latent goes to q_out, the other one into the cache (zero beyond kv_rank). */
typedef struct q38_latent_append_params {
  const void* proj;
  int ld_proj;
  int act;
  int q_rank, kv_rank;
  const float* q_gain;  /* [q_rank] */
  const float* kv_gain; /* [kv_rank] */
  float eps;
  void* q_out;
  int ld_q;
} q38_latent_append_params;
int q38_latent_append(const q38_latent_append_params* p, const q38_batch_desc* batch, const q38_kv_layer_desc* kv, void* stream);
/* Causal softmax attention of `heads` queries per token over the latents: out_h = sum_j softmax_j(scale q_h . c_j) c_j. */
typedef struct q38_latent_attention_params {
  const void* q;        /* [M][heads][k_dim] */
  int act;
  int heads;
  float scale;
  void* out;            /* [M][heads][k_dim] */
  float* partials;      /* scratch for divided key ranges; q38_latent_attention_partial_floats() is always enough */
  size_t partial_floats;
} q38_latent_attention_params;
size_t q38_latent_attention_partial_floats(int k_dim);
int q38_latent_attention(const q38_latent_attention_params* p, const q38_batch_desc* batch, const q38_kv_layer_desc* kv,
                         void* stream);

/* Attention over packed keys and values (bf16, prefill steps): the contexts (positions 0 ... pos0 + count - 1) of the batch's
 * sequences one after the other, each rounded up to whole pages of 64 rows; `rows` is their sum.
 * Gather: the cached latents [rows][k_dim], zero behind a context's end. */
int q38_latent_gather(const q38_batch_desc* batch, const q38_kv_layer_desc* kv, int max_context, int rows, void* out,
                      void* stream);
/* Causal softmax attention, head h of a query, key or value at column h * its stride, zero-padded to a multiple of 16; the
 * output is multiplied by sigmoid(gate) unless gate is NULL. */
typedef struct q38_packed_attention_params {
  const void* q; /* [M][ld_q] */
  int ld_q, q_stride;
  const void *k, *v; /* [rows][ld_kv] */
  int ld_kv, k_stride, v_stride;
  int heads, dim, vdim;
  float scale;
  const void* gate; /* [M][ld_gate]: heads x vdim, or NULL */
  int ld_gate;
  void* out; /* [M][ld_out]: heads x vdim */
  int ld_out;
} q38_packed_attention_params;
int q38_packed_attention_fits(int dim, int vdim);
int q38_packed_attention(const q38_packed_attention_params* p, const q38_batch_desc* batch, void* stream);

/* Diagnostics. */
const char* q38_last_error(void);           /* message of the last failed launcher call on this thread */
/* Programmatic dependent launch (on by default): every launcher allows its kernel to be scheduled while the
 * previous kernel of the stream drains; inside, griddepcontrol.wait precedes the first access to data an earlier
 * kernel produces, so results do not depend on the setting. Off = classic stream order. Applies to launches (and
 * graph captures) made after the call. No counterpart in the reference. */
void q38_set_dependent_launch(int allowed);
unsigned int q38_device_error(int clear);   /* non-zero if a bounded device-side wait ran out (synchronises) */
/* The same status without a synchronisation, as one more node of the caller's stream or graph: a one-thread kernel
 * moves the first non-zero error word of the library into *dst (device memory or mapped pinned host memory) and
 * clears the library's words; *dst is not written when nothing failed. A host engine enqueues it at the end of each
 * step and reads *dst after its stream synchronisation: a step whose pipeline aborted (the results of that launch
 * are meaningless) can then be failed instead of delivered. The first call on a device looks the words up and
 * should come before any stream capture. No counterpart in the reference (its kernels have no bounded waits). */
int q38_device_error_collect(unsigned int* dst, void* stream);
/* Test hook: sets one of the library's error words from the host, as if a kernel had reported `code`. */
int q38_device_error_inject(unsigned int code);
int q38_num_sms(void);                      /* SM count of the current device as cached by the library */

#ifdef __cplusplus
}
#endif
#endif /* Q38_KERNELS_H_ */
