// Attention of the layer-list architectures, general part: rotary positions + value blending + cache append, and the
// head-mixing attention for any head count, head size and precision on the CUDA cores. The bf16 tensor-core kernels that
// serve the usual shapes are in mixed_attention_mma.cu; fp32 runs and outsized shapes come here.
//
// The heads' softmax weights are mixed before they meet the values, so a head's normaliser must be known before any of
// its weights is used: one kernel finds (maximum, 1 / sum) per (token, head), a second one recomputes the scores,
// normalises, mixes over the heads in shared memory and accumulates the values.
#include <algorithm>

#include "act.cuh"
#include "mixed_attention.h"

namespace q38 {
Q38_REGISTER_ERROR_WORD();
namespace {

template <typename T>
__device__ __forceinline__ const T* k_row(const q38_kv_layer_desc& kv, int page, int head, int tok) {
  return reinterpret_cast<const T*>(kv.pages + (size_t)page * kv.page_bytes) + ((size_t)head * Q38_PAGE_TOKENS + tok) * kv.k_dim;
}
template <typename T>
__device__ __forceinline__ const T* v_col(const q38_kv_layer_desc& kv, int page, int head, int d) {
  return reinterpret_cast<const T*>(kv.pages + (size_t)page * kv.page_bytes) +
         (size_t)kv.kv_heads * Q38_PAGE_TOKENS * kv.k_dim + ((size_t)head * kv.v_dim + d) * Q38_PAGE_TOKENS;
}

// ---- rotary positions, value blending, append ------------------------------------------------------------------------
// One CTA per token. The angle position * inv_freq[i] is formed and reduced in double precision, so that far
// positions keep the accuracy of near ones; its sine and cosine are fp32.
template <typename T>
__global__ void __launch_bounds__(256) rope_append_kernel(q38_rope_append_params p, q38_batch_desc b, q38_kv_layer_desc kv) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ float trig[];  // [rot_dims / 2][cos, sin]
  const int m = blockIdx.x, pos = b.tok_pos[m], slot = b.seq_slot[b.tok_seq[m]];
  const int half = p.rot_dims / 2;
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    const double ang = double(pos) * p.inv_freq[i];
    const double turns = ang * 0.15915494309189535;
    const float red = float((turns - rint(turns)) * 6.283185307179586);
    float sn, cs;
    sincosf(red, &sn, &cs);
    trig[2 * i] = cs;
    trig[2 * i + 1] = sn;
  }
  __syncthreads();
  const T* row = static_cast<const T*>(p.proj) + (size_t)m * p.ld_proj;
  const int page = kv.block_table[(size_t)slot * kv.max_pages_per_seq + pos / Q38_PAGE_TOKENS], at = pos % Q38_PAGE_TOKENS;
  if (page < 0 || page >= kv.num_pages) {
    report_error(0x701);
    return;
  }
  uint8_t* base = kv.pages + (size_t)page * kv.page_bytes;
  // one warp per query or key head
  auto turn_head = [&](const T* h, T* out) {
    for (int d = threadIdx.x & 31; d < kv.k_dim; d += 32) {
      float y = 0.0f;
      if (d < p.dim) {
        y = to_f32(h[d]);
        if (d < 2 * half) {
          const int i = d < half ? d : d - half;
          const float cs = trig[2 * i], sn = trig[2 * i + 1];
          y = d < half ? y * cs - to_f32(h[d + half]) * sn : y * cs + to_f32(h[d - half]) * sn;
        }
      }
      out[d] = from_f32<T>(y);
    }
  };
  const int warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  T* q = static_cast<T*>(p.q_out) + (size_t)m * p.heads * kv.k_dim;
  const T* krow = row + (size_t)p.heads * p.dim;
  for (int h = warp; h < p.heads + p.kv_heads; h += warps) {
    const bool key = h >= p.heads;
    turn_head(row + (size_t)h * p.dim, key ? reinterpret_cast<T*>(base) + ((size_t)(h - p.heads) * Q38_PAGE_TOKENS + at) * kv.k_dim
                                           : q + (size_t)h * kv.k_dim);
  }
  const T* vrow = krow + (size_t)p.kv_heads * p.dim;
  T* vbase = reinterpret_cast<T*>(base) + (size_t)p.kv_heads * Q38_PAGE_TOKENS * kv.k_dim;
  const T* first_in = static_cast<const T*>(p.v_first_in);
  T* first_out = static_cast<T*>(p.v_first_out);
  const float lam = first_in ? *p.v_mix : 0.0f;
  const size_t vw = (size_t)p.kv_heads * p.vdim;
  for (int h = warp; h < p.kv_heads; h += warps)
    for (int d = threadIdx.x & 31; d < kv.v_dim; d += 32) {
      float v = 0.0f;
      if (d < p.vdim) {
        const size_t c = (size_t)h * p.vdim + d;
        v = to_f32(vrow[c]);
        if (first_out) first_out[(size_t)m * vw + c] = from_f32<T>(v);
        if (first_in) v = (1.0f - lam) * v + lam * to_f32(first_in[(size_t)m * vw + c]);
      }
      vbase[((size_t)h * kv.v_dim + d) * Q38_PAGE_TOKENS + at] = from_f32<T>(v);
    }
}

// ---- general attention ---------------------------------------------------------------------------------------------------
template <typename T>
__device__ __forceinline__ float dot_row(const float* q, const T* k, int n);
template <>
__device__ __forceinline__ float dot_row<float>(const float* q, const float* k, int n) {
  float s = 0.0f;
  for (int d = 0; d < n; d += 4) {
    const float4 a = *reinterpret_cast<const float4*>(q + d), b = *reinterpret_cast<const float4*>(k + d);
    s += a.x * b.x + a.y * b.y + a.z * b.z + a.w * b.w;
  }
  return s;
}
template <>
__device__ __forceinline__ float dot_row<__nv_bfloat16>(const float* q, const __nv_bfloat16* k, int n) {
  float s = 0.0f;
  for (int d = 0; d < n; d += 8) {
    const uint4 raw = *reinterpret_cast<const uint4*>(k + d);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 f = __bfloat1622float2(h[i]);
      s += q[d + 2 * i] * f.x + q[d + 2 * i + 1] * f.y;
    }
  }
  return s;
}

// (maximum, 1 / sum of exponentials) of one (token, head)
template <typename T>
__global__ void __launch_bounds__(128) mixed_stats_kernel(q38_mixed_attention_params p, q38_batch_desc b, q38_kv_layer_desc kv) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ float q_sm[];
  __shared__ float red_m[4], red_l[4];
  const int i = blockIdx.x, h = blockIdx.y, row = b.seq_start[0] + i;
  const int pos = b.tok_pos[i], slot = b.seq_slot[b.tok_seq[i] - b.tok_seq[0]];
  const int g = h / (p.heads / kv.kv_heads), lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const T* q = static_cast<const T*>(p.q) + ((size_t)row * p.heads + h) * kv.k_dim;
  for (int d = threadIdx.x; d < kv.k_dim; d += blockDim.x) q_sm[d] = to_f32(q[d]);
  __syncthreads();
  const int* table = kv.block_table + (size_t)slot * kv.max_pages_per_seq;
  float mx = -INFINITY, l = 0.0f;
  for (int j = threadIdx.x; j <= pos; j += blockDim.x) {
    const float s = dot_row<T>(q_sm, k_row<T>(kv, table[j / Q38_PAGE_TOKENS], g, j % Q38_PAGE_TOKENS), kv.k_dim) * p.scale;
    const float nm = fmaxf(mx, s);
    l = l * expf(mx - nm) + expf(s - nm);
    mx = nm;
  }
  float M = warp_max(mx);
  l = warp_sum(mx == -INFINITY ? 0.0f : l * expf(mx - M));
  if (lane == 0) {
    red_m[warp] = M;
    red_l[warp] = l;
  }
  __syncthreads();
  if (threadIdx.x == 0) {
    M = fmaxf(fmaxf(red_m[0], red_m[1]), fmaxf(red_m[2], red_m[3]));
    float total = 0.0f;
    for (int w = 0; w < 4; ++w)
      if (red_m[w] != -INFINITY) total += red_l[w] * expf(red_m[w] - M);
    p.stats[((size_t)row * p.heads + h) * 2] = M;
    p.stats[((size_t)row * p.heads + h) * 2 + 1] = 1.0f / total;
  }
}

constexpr int kGenKeys = 32;
template <typename T>
__global__ void __launch_bounds__(256) mixed_values_kernel(q38_mixed_attention_params p, q38_batch_desc b, q38_kv_layer_desc kv) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ float sm[];
  float* q_sm = sm;                                // [H][k_dim]
  float* w_sm = q_sm + p.heads * kv.k_dim;         // [H][keys] softmax weights
  float* x_sm = w_sm + p.heads * kGenKeys;         // [H][keys] mixed weights
  float* acc = x_sm + p.heads * kGenKeys;          // [H][v_dim]
  const int i = blockIdx.x, row = b.seq_start[0] + i, H = p.heads;
  const int pos = b.tok_pos[i], slot = b.seq_slot[b.tok_seq[i] - b.tok_seq[0]], group = H / kv.kv_heads;
  const T* q = static_cast<const T*>(p.q) + (size_t)row * H * kv.k_dim;
  for (int d = threadIdx.x; d < H * kv.k_dim; d += blockDim.x) q_sm[d] = to_f32(q[d]);
  for (int d = threadIdx.x; d < H * kv.v_dim; d += blockDim.x) acc[d] = 0.0f;
  __syncthreads();
  const int* table = kv.block_table + (size_t)slot * kv.max_pages_per_seq;
  const float* stats = p.stats + (size_t)row * H * 2;
  for (int j0 = 0; j0 <= pos; j0 += kGenKeys) {
    const int page = table[j0 / Q38_PAGE_TOKENS], in_page = j0 % Q38_PAGE_TOKENS;
    for (int e = threadIdx.x; e < H * kGenKeys; e += blockDim.x) {
      const int h = e / kGenKeys, j = e % kGenKeys;
      float w = 0.0f;
      if (j0 + j <= pos) {
        const float s = dot_row<T>(q_sm + h * kv.k_dim, k_row<T>(kv, page, h / group, in_page + j), kv.k_dim) * p.scale;
        w = expf(s - stats[2 * h]) * stats[2 * h + 1];
      }
      w_sm[e] = w;
    }
    __syncthreads();
    const float* use = w_sm;
    if (p.head_mix) {
      for (int e = threadIdx.x; e < H * kGenKeys; e += blockDim.x) {
        const int h = e / kGenKeys, j = e % kGenKeys;
        float x = 0.0f;
        for (int g = 0; g < H; ++g) x += p.head_mix[h * H + g] * w_sm[g * kGenKeys + j];
        x_sm[e] = x;
      }
      use = x_sm;
      __syncthreads();
    }
    for (int e = threadIdx.x; e < H * kv.v_dim; e += blockDim.x) {
      const int h = e / kv.v_dim, d = e % kv.v_dim;
      const T* v = v_col<T>(kv, page, h / group, d) + in_page;
      const float* w = use + h * kGenKeys;
      float s = acc[e];
#pragma unroll 8
      for (int j = 0; j < kGenKeys; ++j) s += w[j] * to_f32(v[j]);
      acc[e] = s;
    }
    __syncthreads();
  }
  T* out = static_cast<T*>(p.out) + (size_t)row * p.ld_out;
  for (int e = threadIdx.x; e < H * p.vdim; e += blockDim.x) {
    const int h = e / p.vdim, d = e % p.vdim;
    out[e] = from_f32<T>(acc[h * kv.v_dim + d]);
  }
}

template <typename T>
int launch_general(const q38_mixed_attention_params& p, const q38_batch_desc& b, const q38_kv_layer_desc& kv, cudaStream_t s) {
  const size_t smem = (size_t(p.heads) * (kv.k_dim + kv.v_dim) + 2 * size_t(p.heads) * kGenKeys) * 4;
  Q38_REQUIRE(smem <= size_t(max_optin_smem()), "mixed_attention: %d heads of %d + %d need %zu bytes of shared memory", p.heads,
              kv.k_dim, kv.v_dim, smem);
  Q38_CUDA_OK(cudaFuncSetAttribute(mixed_values_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, max_optin_smem()));
  (void)launch_kernel(mixed_stats_kernel<T>, dim3(b.num_tokens, p.heads), dim3(128), size_t(kv.k_dim) * 4, s, p, b, kv);
  Q38_LAUNCH_OK("mixed_stats_kernel");
  (void)launch_kernel(mixed_values_kernel<T>, dim3(b.num_tokens), dim3(256), smem, s, p, b, kv);
  Q38_LAUNCH_OK("mixed_values_kernel");
  return Q38_OK;
}

int check_attention(const q38_mixed_attention_params* p, const q38_batch_desc* b, const q38_kv_layer_desc* kv) {
  Q38_REQUIRE(p && b && kv && p->q && p->out && p->stats && kv->pages && kv->block_table, "mixed_attention: null argument");
  Q38_REQUIRE(kv->kv_heads > 0 && p->heads > 0 && p->heads % kv->kv_heads == 0, "mixed_attention: heads %d / %d", p->heads, kv->kv_heads);
  Q38_REQUIRE(kv->k_dim % 32 == 0 && kv->v_dim % 8 == 0 && p->vdim > 0 && p->vdim <= kv->v_dim, "mixed_attention: head sizes");
  Q38_REQUIRE(kv->dtype == (p->act == Q38_ACT_BF16 ? Q38_KV_BF16 : Q38_KV_F32), "mixed_attention: cache precision %d", kv->dtype);
  Q38_REQUIRE(p->ld_out >= p->heads * p->vdim, "mixed_attention: ld_out");
  return Q38_OK;
}

}  // namespace
}  // namespace q38

using namespace q38;

extern "C" int q38_rope_append(const q38_rope_append_params* p, const q38_batch_desc* batch, const q38_kv_layer_desc* kv,
                               void* stream) {
  Q38_REQUIRE(p && batch && kv && p->proj && p->q_out && kv->pages && kv->block_table, "rope_append: null argument");
  if (batch->num_tokens == 0) return Q38_OK;
  Q38_REQUIRE(p->heads > 0 && p->kv_heads == kv->kv_heads && p->dim <= kv->k_dim && p->vdim <= kv->v_dim, "rope_append: sizes");
  Q38_REQUIRE(p->rot_dims >= 0 && p->rot_dims % 2 == 0 && p->rot_dims <= p->dim && p->rot_dims <= 4096, "rope_append: rot_dims %d", p->rot_dims);
  Q38_REQUIRE(p->ld_proj >= p->heads * p->dim + p->kv_heads * (p->dim + p->vdim), "rope_append: ld_proj");
  Q38_REQUIRE(kv->dtype == (p->act == Q38_ACT_BF16 ? Q38_KV_BF16 : Q38_KV_F32), "rope_append: cache precision");
  Q38_REQUIRE(p->rot_dims == 0 || p->inv_freq, "rope_append: inv_freq");
  Q38_REQUIRE(!p->v_first_in || p->v_mix, "rope_append: v_mix");
  const size_t smem = size_t(std::max(1, p->rot_dims)) * 4;
  if (p->act == Q38_ACT_BF16)
    (void)launch_kernel(rope_append_kernel<__nv_bfloat16>, dim3(batch->num_tokens), dim3(256), smem, as_stream(stream), *p, *batch, *kv);
  else
    (void)launch_kernel(rope_append_kernel<float>, dim3(batch->num_tokens), dim3(256), smem, as_stream(stream), *p, *batch, *kv);
  Q38_LAUNCH_OK("rope_append_kernel");
  return Q38_OK;
}

extern "C" int q38_mixed_attention_prefill(const q38_mixed_attention_params* p, const q38_batch_desc* batch,
                                           const q38_kv_layer_desc* kv, void* stream) {
  if (const int rc = check_attention(p, batch, kv)) return rc;
  if (batch->num_tokens == 0) return Q38_OK;
  if (p->act == Q38_ACT_F32) return launch_general<float>(*p, *batch, *kv, as_stream(stream));
  if (mixed_prefill_mma_fits(*p, *kv)) return mixed_prefill_mma(*p, *batch, *kv, as_stream(stream));
  return launch_general<__nv_bfloat16>(*p, *batch, *kv, as_stream(stream));
}

extern "C" int q38_mixed_attention_decode(const q38_mixed_attention_params* p, const q38_batch_desc* batch,
                                          const q38_kv_layer_desc* kv, void* stream) {
  if (const int rc = check_attention(p, batch, kv)) return rc;
  if (batch->num_tokens == 0) return Q38_OK;
  if (p->act == Q38_ACT_F32) return launch_general<float>(*p, *batch, *kv, as_stream(stream));
  if (batch->num_tokens == batch->num_seqs && mixed_decode_mma_fits(*p, *kv)) return mixed_decode_mma(*p, *batch, *kv, as_stream(stream));
  return launch_general<__nv_bfloat16>(*p, *batch, *kv, as_stream(stream));
}
