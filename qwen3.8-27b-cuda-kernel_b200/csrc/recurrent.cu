// Elementwise gated linear recurrences of the layer-list architectures: minGRU and the RG-LRU behind a causal
// convolution. Both are S_t = a_t S_(t-1) + b_t per channel; they differ in how a and b come about and in what leaves.
//
// Prefill: one CTA per (32 channels, sequence). 32 time segments of up to 8 tokens each run side by side: a thread
// computes its segment's (a, b) in registers, scans them locally, takes the state that enters its segment from the
// segment totals in shared memory, and emits. Decode batches: one thread per (sequence, channel).
// The RG-LRU's a and b need a block-diagonal product of the convolved inputs with bf16 matrices. With bf16 activations
// that product runs on mma.sync with the fp32 convolution output split into two bf16 terms (hi + lo, 16 mantissa bits),
// with fp32 activations on the CUDA cores.
#include <algorithm>

#include "act.cuh"
#include "host_util.h"

namespace q38 {
Q38_REGISTER_ERROR_WORD();
namespace {

constexpr int kScanCh = 32, kScanSegs = 32, kSegTokens = 8;

struct Row {  // one sequence's run in this step
  int start, count, pos0, slot;
};
__device__ __forceinline__ Row row_of(const q38_batch_desc& b, int s) {
  return {b.seq_start[s], b.seq_start[s + 1] - b.seq_start[s], b.seq_pos0[s], b.seq_slot[s]};
}

// ---- minGRU ---------------------------------------------------------------------------------------------------
template <typename T>
struct MinGru {
  q38_mingru_params p;
  __device__ __forceinline__ void coeffs(int t, int c, float& a, float& b) const {
    const T* r = static_cast<const T*>(p.proj) + (size_t)t * p.ld_proj;
    const float z = sigmoid_f(to_f32(r[c])), u = to_f32(r[p.width + c]);
    const float cand = u >= 0.0f ? u + 0.5f : sigmoid_f(u);
    a = 1.0f - z;
    b = z * cand;
  }
  __device__ __forceinline__ void emit(int t, int c, float S) const {
    const T* r = static_cast<const T*>(p.proj) + (size_t)t * p.ld_proj;
    static_cast<T*>(p.out)[(size_t)t * p.ld_out + c] = from_f32<T>(S * silu_f(to_f32(r[2 * p.width + c])));
  }
  __device__ __forceinline__ void finish(const Row&, int, const q38_recurrent_state_desc&) const {}
};

// ---- RG-LRU (a and b from the gate kernel's scratch) -------------------------------------------------------------
template <typename T>
struct RgLru {
  q38_rglru_params p;
  q38_batch_desc batch;
  __device__ __forceinline__ void coeffs(int t, int c, float& a, float& b) const {
    const size_t i = size_t(t - batch.seq_start[0]);
    a = p.scratch[i * p.width + c];
    b = p.scratch[((size_t)batch.num_tokens + i) * p.width + c];
  }
  __device__ __forceinline__ void emit(int t, int c, float S) const {
    const T* r = static_cast<const T*>(p.proj) + (size_t)t * p.ld_proj;
    static_cast<T*>(p.out)[(size_t)t * p.ld_out + c] = from_f32<T>(S * gelu_tanh_f(to_f32(r[c])));
  }
  // the run's last inputs into the convolution ring (one thread per channel; the gate kernel is complete)
  __device__ __forceinline__ void finish(const Row& row, int c, const q38_recurrent_state_desc& st) const {
    T* ring = reinterpret_cast<T*>(st.conv + (size_t)row.slot * st.slot_bytes);
    for (int i = max(0, row.count - p.taps); i < row.count; ++i)
      ring[(size_t)((row.pos0 + i) % p.taps) * p.width + c] =
          static_cast<const T*>(p.proj)[(size_t)(row.start + i) * p.ld_proj + p.width + c];
  }
};

template <typename Op>
__global__ void __launch_bounds__(kScanCh * kScanSegs)
scan_kernel(Op op, int width, q38_batch_desc batch, q38_recurrent_state_desc st) {
  pdl_wait();
  pdl_launch_dependents();
  __shared__ float ta[kScanSegs][kScanCh], tb[kScanSegs][kScanCh];
  const int lane = threadIdx.x, seg = threadIdx.y;
  const int c = blockIdx.x * kScanCh + lane;
  const bool live = c < width;
  const Row row = row_of(batch, blockIdx.y);
  float* state = reinterpret_cast<float*>(st.state + (size_t)row.slot * st.slot_bytes);
  float S = live && row.pos0 > 0 ? state[c] : 0.0f;  // the state that enters the current token block
  for (int base = 0; base < row.count; base += kScanSegs * kSegTokens) {
    const int n = min(kScanSegs * kSegTokens, row.count - base);
    const int len = (n + kScanSegs - 1) / kScanSegs;
    const int lo = min(n, seg * len), hi = min(n, lo + len);
    float a[kSegTokens], b[kSegTokens];
    float A = 1.0f, B = 0.0f;
#pragma unroll
    for (int i = 0; i < kSegTokens; ++i) {
      a[i] = 1.0f;
      b[i] = 0.0f;
      if (live && lo + i < hi) op.coeffs(row.start + base + lo + i, c, a[i], b[i]);
    }
#pragma unroll
    for (int i = 0; i < kSegTokens; ++i) {
      A *= a[i];
      B = a[i] * B + b[i];
    }
    ta[seg][lane] = A;
    tb[seg][lane] = B;
    __syncthreads();
    float s = S;
    for (int k = 0; k < seg; ++k) s = ta[k][lane] * s + tb[k][lane];
    float total = s;
    for (int k = seg; k < kScanSegs; ++k) total = ta[k][lane] * total + tb[k][lane];
#pragma unroll
    for (int i = 0; i < kSegTokens; ++i) {
      s = a[i] * s + b[i];
      if (live && lo + i < hi) op.emit(row.start + base + lo + i, c, s);
    }
    S = total;
    __syncthreads();
  }
  if (live && seg == 0 && row.count > 0) {
    state[c] = S;
    op.finish(row, c, st);
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
mingru_decode_kernel(MinGru<T> op, int width, q38_batch_desc batch, q38_recurrent_state_desc st) {
  pdl_wait();
  pdl_launch_dependents();
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= width) return;
  const Row row = row_of(batch, blockIdx.y);
  float* state = reinterpret_cast<float*>(st.state + (size_t)row.slot * st.slot_bytes);
  float a, b;
  op.coeffs(row.start, c, a, b);
  const float S = (row.pos0 > 0 ? a * state[c] : 0.0f) + b;
  state[c] = S;
  op.emit(row.start, c, S);
}

// ---- RG-LRU gates -------------------------------------------------------------------------------------------------
// u = conv(x) of one (token, channel); token i of the (sub-)batch is row seq_start[0] + i of the step. Inputs of this step from proj, older ones from the slot's ring, none before the
// sequence's start.
template <typename T>
__device__ __forceinline__ float conv_at(const q38_rglru_params& p, const q38_batch_desc& b, const uint8_t* conv,
                                         size_t slot_bytes, int i, int c) {
  const int s = b.tok_seq[i] - b.tok_seq[0], pos = b.tok_pos[i], pos0 = b.seq_pos0[s], t = b.seq_start[0] + i;
  const T* x = static_cast<const T*>(p.proj) + p.width + c;
  const T* ring = reinterpret_cast<const T*>(conv + (size_t)b.seq_slot[s] * slot_bytes);
  float u = p.conv_b[c];
  for (int j = 0; j < p.taps; ++j) {
    const int q = pos - (p.taps - 1 - j);
    if (q < 0) continue;
    const float v = q >= pos0 ? to_f32(x[(size_t)(t - (pos - q)) * p.ld_proj]) : to_f32(ring[(size_t)(q % p.taps) * p.width + c]);
    u += p.conv_w[(size_t)j * p.width + c] * v;
  }
  return u;
}

struct GateConst {  // of one channel: the gates' biases and log_decay * softplus(lam)
  float rb, ib, decay;
};
__device__ __forceinline__ GateConst gate_const(const q38_rglru_params& p, int c) {
  return {p.gate_b[c], p.gate_b[p.width + c], p.log_decay * softplus_f(p.lam[c])};
}

// From the gates' pre-activations to (a, b); decode batches go on to the state and the output.
template <typename T, bool DECODE>
__device__ __forceinline__ void gate_finish(const q38_rglru_params& p, const q38_batch_desc& b,
                                            const q38_recurrent_state_desc& st, int i, int c, float r_pre, float i_pre, float u,
                                            const GateConst& k) {
  const int t = b.seq_start[0] + i;
  const float r = sigmoid_f(r_pre + k.rb), gi = sigmoid_f(i_pre + k.ib);
  const float log_a = k.decay * r;
  const float a = expf(log_a);
  const float x = sqrtf(-expm1f(2.0f * log_a)) * gi * u;
  if (!DECODE) {
    p.scratch[(size_t)i * p.width + c] = a;
    p.scratch[((size_t)b.num_tokens + i) * p.width + c] = x;
    return;
  }
  const int slot = b.seq_slot[b.tok_seq[i] - b.tok_seq[0]], pos = b.tok_pos[i];
  float* state = reinterpret_cast<float*>(st.state + (size_t)slot * st.slot_bytes);
  const float S = (pos > 0 ? a * state[c] : 0.0f) + x;
  state[c] = S;
  const T* row = static_cast<const T*>(p.proj) + (size_t)t * p.ld_proj;
  // this token's input takes the ring row of position pos - taps, which no other CTA of this launch reads
  reinterpret_cast<T*>(st.conv + (size_t)slot * st.slot_bytes)[(size_t)(pos % p.taps) * p.width + c] = row[p.width + c];
  static_cast<T*>(p.out)[(size_t)t * p.ld_out + c] = from_f32<T>(S * gelu_tanh_f(to_f32(row[c])));
}

constexpr int kGateTokens = 8, kGateThreads = 128;
// CUDA-core form: a CTA holds the convolved inputs of 8 tokens x one block; a thread owns one output channel.
template <typename T, bool DECODE>
__global__ void __launch_bounds__(kGateThreads)
rglru_gates_kernel(q38_rglru_params p, q38_batch_desc batch, q38_recurrent_state_desc st) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ float u_sm[];  // [kGateTokens][block_ld]
  const int bs = p.width / p.blocks, blk = blockIdx.y, t0 = blockIdx.x * kGateTokens;
  const int n = min(kGateTokens, batch.num_tokens - t0);
  for (int i = threadIdx.x; i < kGateTokens * p.block_ld; i += blockDim.x) {
    const int t = i / p.block_ld, k = i % p.block_ld;
    float u = 0.0f;
    if (t < n && k < bs) u = conv_at<T>(p, batch, st.conv, st.slot_bytes, t0 + t, blk * bs + k);
    u_sm[i] = u;
  }
  __syncthreads();
  const __nv_bfloat16* wr = reinterpret_cast<const __nv_bfloat16*>(p.gate_w) + (size_t)blk * 2 * p.block_ld * p.block_ld;
  const __nv_bfloat16* wi = wr + (size_t)p.block_ld * p.block_ld;
  for (int o = threadIdx.x + blockIdx.z * blockDim.x; o < bs; o += blockDim.x * gridDim.z) {
    float ar[kGateTokens] = {}, ai[kGateTokens] = {};
    for (int k = 0; k < p.block_ld; k += 2) {
      const float2 r2 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(wr + (size_t)o * p.block_ld + k));
      const float2 i2 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(wi + (size_t)o * p.block_ld + k));
#pragma unroll
      for (int t = 0; t < kGateTokens; ++t) {
        const float2 u = *reinterpret_cast<const float2*>(u_sm + t * p.block_ld + k);
        ar[t] += r2.x * u.x + r2.y * u.y;
        ai[t] += i2.x * u.x + i2.y * u.y;
      }
    }
    for (int t = 0; t < n; ++t) {
      float r = 0, gi = 0;
#pragma unroll
      for (int q = 0; q < kGateTokens; ++q)
        if (q == t) r = ar[q], gi = ai[q];
      gate_finish<T, DECODE>(p, batch, st, t0 + t, blk * bs + o, r, gi, u_sm[t * p.block_ld + o], gate_const(p, blk * bs + o));
    }
  }
}

// Tensor-core form (bf16 activations): a CTA holds the convolved inputs of 32 tokens x one block in shared memory, as
// bf16 terms hi + lo, and makes output channels of both gates, 64 at a time: a warp the 8 channels of one n tile, r and i
// side by side in its registers. Weights come straight from global memory into fragments (16 contiguous bytes of a row = two k16
// steps under a permutation of k that both operands share).
constexpr int kMmaTokens = 32, kMmaWarps = 8, kMmaOut = kMmaWarps * 8;
__host__ __device__ constexpr int gate_stride(int cols) { return cols % 64 == 32 ? cols : cols + 32; }

template <bool DECODE>
__global__ void __launch_bounds__(kMmaWarps * 32)
rglru_gates_mma_kernel(q38_rglru_params p, q38_batch_desc batch, q38_recurrent_state_desc st) {
  extern __shared__ __align__(16) uint8_t smem[];
  const int bs = p.width / p.blocks, ld = p.block_ld, us = gate_stride(ld), blk = blockIdx.y, t0 = blockIdx.x * kMmaTokens;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
  __nv_bfloat16* hi = reinterpret_cast<__nv_bfloat16*>(smem);  // [32][us]
  __nv_bfloat16* lo = hi + kMmaTokens * us;
  const __nv_bfloat16* gw = reinterpret_cast<const __nv_bfloat16*>(p.gate_w) + ((size_t)blk * 2 * ld + g) * ld + t * 8;
  pdl_wait();
  pdl_launch_dependents();
  const int n = min(kMmaTokens, batch.num_tokens - t0);
  __shared__ int tok_pos[kMmaTokens], tok_pos0[kMmaTokens];
  __shared__ const __nv_bfloat16* tok_ring[kMmaTokens];
  if (threadIdx.x < n) {
    const int s = batch.tok_seq[t0 + threadIdx.x] - batch.tok_seq[0];
    tok_pos[threadIdx.x] = batch.tok_pos[t0 + threadIdx.x];
    tok_pos0[threadIdx.x] = batch.seq_pos0[s];
    tok_ring[threadIdx.x] = reinterpret_cast<const __nv_bfloat16*>(st.conv + (size_t)batch.seq_slot[s] * st.slot_bytes);
  }
  __syncthreads();
  const __nv_bfloat16* x0 = static_cast<const __nv_bfloat16*>(p.proj) + (size_t)(batch.seq_start[0] + t0) * p.ld_proj + p.width;
  if (bs % 8 == 0 && p.width % 8 == 0 && p.ld_proj % 8 == 0 && p.taps <= 4) {
    // a thread keeps the taps of eight channels in registers and takes several tokens; all inputs of a token are
    // requested before the first is used
    const int vecs = ld / 8;
    for (int kv = threadIdx.x & 31; kv < vecs; kv += 32) {
      const int k = kv * 8, c = blk * bs + k;
      const bool in_block = k < bs;
      float w[4][8], bias[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        bias[e] = in_block ? p.conv_b[c + e] : 0.0f;
#pragma unroll
        for (int j = 0; j < 4; ++j) w[j][e] = in_block && j < p.taps ? p.conv_w[(size_t)(p.taps - 1 - j) * p.width + c + e] : 0.0f;
      }
      for (int tok = warp; tok < kMmaTokens; tok += kMmaWarps) {
        float u[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) u[e] = bias[e];
        uint4 in[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {  // j tokens back
          in[j] = make_uint4(0, 0, 0, 0);
          if (in_block && tok < n && j < p.taps) {
            const int q = tok_pos[tok] - j;
            if (q >= tok_pos0[tok]) in[j] = *reinterpret_cast<const uint4*>(x0 + (ptrdiff_t)(tok - j) * p.ld_proj + c);
            else if (q >= 0) in[j] = *reinterpret_cast<const uint4*>(tok_ring[tok] + (size_t)(q % p.taps) * p.width + c);
          }
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const __nv_bfloat162* v = reinterpret_cast<const __nv_bfloat162*>(&in[j]);
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float2 f = __bfloat1622float2(v[e]);
            u[2 * e] += w[j][2 * e] * f.x;
            u[2 * e + 1] += w[j][2 * e + 1] * f.y;
          }
        }
        __nv_bfloat162 h[4], l[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          h[e] = __floats2bfloat162_rn(u[2 * e], u[2 * e + 1]);
          const float2 f = __bfloat1622float2(h[e]);
          l[e] = __floats2bfloat162_rn(u[2 * e] - f.x, u[2 * e + 1] - f.y);
        }
        *reinterpret_cast<uint4*>(hi + tok * us + k) = *reinterpret_cast<const uint4*>(h);
        *reinterpret_cast<uint4*>(lo + tok * us + k) = *reinterpret_cast<const uint4*>(l);
      }
    }
  } else {
    for (int i = threadIdx.x; i < kMmaTokens * ld; i += blockDim.x) {
      const int tok = i / ld, k = i % ld;
      const float u = tok < n && k < bs ? conv_at<__nv_bfloat16>(p, batch, st.conv, st.slot_bytes, t0 + tok, blk * bs + k) : 0.0f;
      const __nv_bfloat16 h = __float2bfloat16_rn(u);
      hi[tok * us + k] = h;
      lo[tok * us + k] = __float2bfloat16_rn(u - __bfloat162float(h));
    }
  }
  __syncthreads();
  for (int o0 = blockIdx.z * kMmaOut + warp * 8; o0 < ld; o0 += gridDim.z * kMmaOut) {
    const __nv_bfloat16* wr = gw + (size_t)o0 * ld;
    const __nv_bfloat16* wi = wr + (size_t)ld * ld;
    float acc[2][2][4] = {};  // [16-token tile][r, i]
#pragma unroll 4
    for (int k = 0; k < ld; k += 32) {
      const uint4 w[2] = {*reinterpret_cast<const uint4*>(wr + k), *reinterpret_cast<const uint4*>(wi + k)};
#pragma unroll
      for (int mt = 0; mt < 2; ++mt)
#pragma unroll
        for (int term = 0; term < 2; ++term) {
          const __nv_bfloat16* u = (term ? lo : hi) + (mt * 16 + g) * us + k + t * 8;
          const AFragPair a = a_fragments(*reinterpret_cast<const uint4*>(u), *reinterpret_cast<const uint4*>(u + 8 * us));
          mma_pair(acc[mt][0], a, w[0]);
          mma_pair(acc[mt][1], a, w[1]);
        }
    }
#pragma unroll
    for (int d = 0; d < 2; ++d) {
      const int o = o0 + 2 * t + d;
      if (o >= bs) continue;
      const int c = blk * bs + o;
      const GateConst gc = gate_const(p, c);
#pragma unroll
      for (int mt = 0; mt < 2; ++mt)
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
          const int tok = mt * 16 + g + 8 * hf;
          if (tok >= n) continue;
          const float u = __bfloat162float(hi[tok * us + o]) + __bfloat162float(lo[tok * us + o]);
          gate_finish<__nv_bfloat16, DECODE>(p, batch, st, t0 + tok, c, acc[mt][0][2 * hf + d], acc[mt][1][2 * hf + d], u, gc);
        }
    }
  }
}

size_t gates_mma_smem(int block_ld) { return size_t(2) * kMmaTokens * gate_stride(block_ld) * 2; }

template <bool DECODE>
int launch_gates_mma(const q38_rglru_params& p, const q38_batch_desc& b, const q38_recurrent_state_desc& st, cudaStream_t s) {
  const int bs = p.width / p.blocks;
  const size_t smem = gates_mma_smem(p.block_ld);
  static const cudaError_t attr = cudaFuncSetAttribute(rglru_gates_mma_kernel<DECODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, max_optin_smem() - 1024);
  Q38_CUDA_OK(attr);
  // few tokens: the output channels of a block over several CTAs; many: one CTA convolves once for all of them
  const int tiles = (b.num_tokens + kMmaTokens - 1) / kMmaTokens;
  const int slices = std::max(1, std::min((bs + kMmaOut - 1) / kMmaOut, 2 * num_sms() / (tiles * p.blocks)));
  (void)launch_kernel(rglru_gates_mma_kernel<DECODE>, dim3(tiles, p.blocks, slices),
                      dim3(kMmaWarps * 32), smem, s, p, b, st);
  Q38_LAUNCH_OK("rglru_gates_mma_kernel");
  return Q38_OK;
}

int check_common(const q38_batch_desc* b, const q38_recurrent_state_desc* st, const char* what) {
  Q38_REQUIRE(b && st && st->state && b->seq_start && b->seq_slot && b->seq_pos0 && b->tok_pos && b->tok_seq, "%s: null argument", what);
  Q38_REQUIRE(b->num_seqs > 0 && b->num_tokens >= b->num_seqs && b->max_tokens_per_seq > 0, "%s: batch sizes", what);
  return Q38_OK;
}

template <typename T>
int launch_mingru(const q38_mingru_params& p, const q38_batch_desc& b, const q38_recurrent_state_desc& st, cudaStream_t s) {
  MinGru<T> op{p};
  if (b.max_tokens_per_seq == 1)
    (void)launch_kernel(mingru_decode_kernel<T>, dim3((p.width + 255) / 256, b.num_seqs), dim3(256), 0, s, op, p.width, b, st);
  else
    (void)launch_kernel(scan_kernel<MinGru<T>>, dim3((p.width + kScanCh - 1) / kScanCh, b.num_seqs), dim3(kScanCh, kScanSegs), 0,
                        s, op, p.width, b, st);
  Q38_LAUNCH_OK("mingru");
  return Q38_OK;
}

template <typename T>
int launch_gates_simt(const q38_rglru_params& p, const q38_batch_desc& b, const q38_recurrent_state_desc& st, bool decode, cudaStream_t s) {
  const int bs = p.width / p.blocks;
  const dim3 grid((b.num_tokens + kGateTokens - 1) / kGateTokens, p.blocks, (bs + kGateThreads - 1) / kGateThreads);
  const size_t smem = size_t(kGateTokens) * p.block_ld * 4;
  Q38_REQUIRE(smem <= size_t(max_optin_smem()), "rglru: blocks of %d channels", bs);
  static const cudaError_t attr0 = cudaFuncSetAttribute(rglru_gates_kernel<T, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, max_optin_smem());
  static const cudaError_t attr1 = cudaFuncSetAttribute(rglru_gates_kernel<T, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, max_optin_smem());
  Q38_CUDA_OK(attr0);
  Q38_CUDA_OK(attr1);
  if (decode)
    (void)launch_kernel(rglru_gates_kernel<T, true>, grid, dim3(kGateThreads), smem, s, p, b, st);
  else
    (void)launch_kernel(rglru_gates_kernel<T, false>, grid, dim3(kGateThreads), smem, s, p, b, st);
  Q38_LAUNCH_OK("rglru_gates_kernel");
  return Q38_OK;
}

template <typename T>
int launch_rglru(const q38_rglru_params& p, const q38_batch_desc& b, const q38_recurrent_state_desc& st, cudaStream_t s) {
  const bool decode = b.max_tokens_per_seq == 1;
  int rc;
  if (sizeof(T) == 2 && gates_mma_smem(p.block_ld) <= size_t(max_optin_smem() - 1024))
    rc = decode ? launch_gates_mma<true>(p, b, st, s) : launch_gates_mma<false>(p, b, st, s);
  else
    rc = launch_gates_simt<T>(p, b, st, decode, s);
  if (rc) return rc;
  if (decode) return Q38_OK;
  RgLru<T> op{p, b};
  (void)launch_kernel(scan_kernel<RgLru<T>>, dim3((p.width + kScanCh - 1) / kScanCh, b.num_seqs), dim3(kScanCh, kScanSegs), 0, s,
                      op, p.width, b, st);
  Q38_LAUNCH_OK("rglru scan_kernel");
  return Q38_OK;
}

}  // namespace
}  // namespace q38

using namespace q38;

extern "C" int q38_mingru(const q38_mingru_params* p, const q38_batch_desc* batch, const q38_recurrent_state_desc* st,
                          void* stream) {
  Q38_REQUIRE(p && p->proj && p->out, "mingru: null argument");
  if (const int rc = check_common(batch, st, "mingru")) return rc;
  Q38_REQUIRE(p->width > 0 && p->ld_proj >= 3 * p->width && p->ld_out >= p->width, "mingru: sizes");
  return p->act == Q38_ACT_BF16 ? launch_mingru<__nv_bfloat16>(*p, *batch, *st, as_stream(stream))
                                : launch_mingru<float>(*p, *batch, *st, as_stream(stream));
}

extern "C" int q38_rglru(const q38_rglru_params* p, const q38_batch_desc* batch, const q38_recurrent_state_desc* st,
                         void* stream) {
  Q38_REQUIRE(p && p->proj && p->out && p->conv_w && p->conv_b && p->gate_w && p->gate_b && p->lam, "rglru: null argument");
  if (const int rc = check_common(batch, st, "rglru")) return rc;
  Q38_REQUIRE(p->width > 0 && p->blocks > 0 && p->width % p->blocks == 0 && p->taps > 0 && st->conv, "rglru: sizes");
  Q38_REQUIRE(p->ld_proj >= 2 * p->width && p->ld_out >= p->width, "rglru: leading dimensions");
  Q38_REQUIRE(p->block_ld % 32 == 0 && p->block_ld >= p->width / p->blocks, "rglru: block_ld %d", p->block_ld);
  Q38_REQUIRE(batch->max_tokens_per_seq == 1 || p->scratch, "rglru: scratch needed");
  return p->act == Q38_ACT_BF16 ? launch_rglru<__nv_bfloat16>(*p, *batch, *st, as_stream(stream))
                                : launch_rglru<float>(*p, *batch, *st, as_stream(stream));
}
