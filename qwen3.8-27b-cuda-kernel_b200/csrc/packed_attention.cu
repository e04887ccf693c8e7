// Causal softmax attention of a prefill step over packed keys and values: the contexts of the step's sequences one after the
// other, each rounded up to whole pages (64 rows), every head's keys and values in place. Latent attention brings the
// cached latents of a step into that form (q38_latent_gather, then one dense product with the heads' key and value matrices)
// when its runs are long enough to pay for it.
//
// One CTA per (64 query tokens, head, sequence), the longest contexts first: four warps of 16 rows each, 64 keys at a time
// through one buffer for keys and one for values, each refilled (cp.async) while the other is used, so that several CTAs
// share an SM; online softmax in registers (mma.sync, fp32 scores, weights and sums). The weights of a
// tile are the A operand of the value product as they stand, as bf16 hi + lo (16 mantissa bits). The output gate is applied
// as the rows are stored.
#include <algorithm>

#include "act.cuh"
#include "host_util.h"

namespace q38 {
Q38_REGISTER_ERROR_WORD();
namespace {

using bf16 = __nv_bfloat16;
constexpr int kPage = Q38_PAGE_TOKENS, kTile = 64, kThreads = 128;
constexpr float kLog2e = 1.4426950408889634f;
__host__ __device__ constexpr int up16(int x) { return (x + 15) / 16 * 16; }

// the value product takes 32 columns at a time
__host__ __device__ constexpr int value_stride(int vdim) { return (vdim + 31) / 32 * 32 + 8; }

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool real) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(real ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - f.x, b - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}

__device__ __forceinline__ int context_of(const q38_batch_desc& b, int s) { return b.seq_pos0[s] + b.seq_start[s + 1] - b.seq_start[s]; }
// first packed row of sequence `seq`; for whole warps
__device__ __forceinline__ int packed_start(const q38_batch_desc& b, int seq) {
  int rows = 0;
  for (int s = threadIdx.x & 31; s < seq; s += 32) rows += (context_of(b, s) + kPage - 1) / kPage * kPage;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) rows += __shfl_xor_sync(0xffffffffu, rows, o);
  return rows;
}

// One CTA per (page, sequence): latents of one page to their packed rows, zeros behind the context's end.
__global__ void __launch_bounds__(256) latent_gather_kernel(q38_batch_desc b, q38_kv_layer_desc kv, int rows, bf16* __restrict__ out) {
  pdl_wait();
  pdl_launch_dependents();
  const int seq = blockIdx.y, pg = blockIdx.x, context = context_of(b, seq);
  if (pg * kPage >= context) return;
  const int first = packed_start(b, seq) + pg * kPage;
  int page = kv.block_table[(size_t)b.seq_slot[seq] * kv.max_pages_per_seq + pg];
  if (page < 0 || page >= kv.num_pages || first + kPage > rows) {
    if (threadIdx.x == 0) report_error(0x911);
    return;
  }
  const uint4* src = reinterpret_cast<const uint4*>(kv.pages + (size_t)page * kv.page_bytes);
  uint4* dst = reinterpret_cast<uint4*>(out + (size_t)first * kv.k_dim);
  const int pieces = kPage * kv.k_dim / 8, live = min(kPage, context - pg * kPage) * kv.k_dim / 8;
  for (int i = threadIdx.x; i < pieces; i += 256) dst[i] = i < live ? src[i] : make_uint4(0, 0, 0, 0);
}

// NV: 8-column tiles of the output held by a warp
template <int NV>
__global__ void __launch_bounds__(kThreads)
packed_attention_kernel(q38_packed_attention_params p, q38_batch_desc b) {
  extern __shared__ __align__(16) uint8_t smem[];
  const int dk = up16(p.dim), dv = up16(p.vdim), ks = dk + 8, vs = value_stride(p.vdim);  // rows an odd multiple of 16 bytes apart
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const uint32_t q_s = smem_u32(smem), k_s = q_s + uint32_t(kTile * ks) * 2, v_s = k_s + uint32_t(kTile * ks) * 2;
  pdl_wait();
  pdl_launch_dependents();
  const int h = blockIdx.x, seq = blockIdx.z, i0 = (int(gridDim.y) - 1 - int(blockIdx.y)) * kTile;
  const int start = b.seq_start[seq], count = b.seq_start[seq + 1] - start, pos0 = b.seq_pos0[seq];
  if (i0 >= count) return;
  const size_t row0 = size_t(packed_start(b, seq));
  const int tokens = min(kTile, count - i0), tiles = (pos0 + i0 + tokens - 1) / kTile + 1;
  const bf16* K = static_cast<const bf16*>(p.k) + row0 * p.ld_kv + (size_t)h * p.k_stride;
  const bf16* V = static_cast<const bf16*>(p.v) + row0 * p.ld_kv + (size_t)h * p.v_stride;
  const bf16* Q = static_cast<const bf16*>(p.q) + (size_t)(start + i0) * p.ld_q + (size_t)h * p.q_stride;

  // 16-byte pieces of a [64][width] tile, dealt to the threads in order
  auto rows_in = [&](uint32_t dst, int stride, const bf16* src, int ld, int width, int live) {
    const int pieces = width / 8, dr = kThreads / pieces, dk8 = kThreads - dr * pieces;
    int row = tid / pieces, k = tid - row * pieces;
    while (row < kTile) {
      cp_async16(dst + uint32_t(row * stride + 8 * k) * 2, src + (size_t)(row < live ? row : 0) * ld + 8 * k, row < live);
      row += dr;
      k += dk8;
      if (k >= pieces) {
        k -= pieces;
        ++row;
      }
    }
  };
  auto load_k = [&](int t) { rows_in(k_s, ks, K + (size_t)t * kTile * p.ld_kv, p.ld_kv, dk, kTile); };
  auto load_v = [&](int t) { rows_in(v_s, vs, V + (size_t)t * kTile * p.ld_kv, p.ld_kv, dv, kTile); };
  if (dv % 32) {  // columns no head has: their products are never stored, but must not be read from nowhere
    for (int i = tid; i < kTile * 8; i += kThreads)
      *reinterpret_cast<uint32_t*>(smem + (v_s - q_s) + ((i >> 3) * vs + dv + 2 * (i & 7)) * 2) = 0;
  }
  rows_in(q_s, ks, Q, p.ld_q, dk, tokens);
  load_k(0);
  cp_async_commit();
  load_v(0);
  cp_async_commit();

  const int ra = 16 * warp + g, pos_a = pos0 + i0 + ra, pos_b = pos_a + 8;
  const float scale2 = p.scale * kLog2e;
  float m_a = -INFINITY, m_b = -INFINITY, l_a = 0.0f, l_b = 0.0f;
  float o[NV][4];
#pragma unroll
  for (int i = 0; i < NV; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[i][e] = 0.0f;
  const uint32_t q_a = q_s + uint32_t((16 * warp + (lane & 15)) * ks + (lane >> 4) * 8) * 2;
  const uint32_t k_a = k_s + uint32_t(((lane & 7) + ((lane >> 4) << 3)) * ks + ((lane >> 3) & 1) * 8) * 2;
  const uint32_t v_a = v_s + uint32_t(((lane & 7) + (((lane >> 3) & 1) << 3)) * vs + (lane >> 4) * 8) * 2;
  cp_async_wait<1>();
  __syncthreads();  // queries and the first keys have landed

  for (int t = 0; t < tiles; ++t) {
    float s[8][4] = {};
#pragma unroll 4
    for (int k = 0; k < dk; k += 16) {
      uint32_t a[4];
      ldmatrix_x4(a, q_a + k * 2);
#pragma unroll
      for (int kp = 0; kp < 4; ++kp) {
        uint32_t kf[4];
        ldmatrix_x4(kf, k_a + uint32_t(kp * 16 * ks + k) * 2);
        mma_bf16_16816(s[2 * kp], a, kf[0], kf[1]);
        mma_bf16_16816(s[2 * kp + 1], a, kf[2], kf[3]);
      }
    }
#pragma unroll
    for (int kt = 0; kt < 8; ++kt)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[kt][e] *= scale2;
    if (t * kTile + kTile - 1 > pos0 + i0 + 16 * warp) {  // some key of the tile lies behind some row of this warp
#pragma unroll
      for (int kt = 0; kt < 8; ++kt)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int key = t * kTile + 8 * kt + 2 * t4 + e;
          if (key > pos_a) s[kt][e] = -INFINITY;
          if (key > pos_b) s[kt][2 + e] = -INFINITY;
        }
    }
    float ma = -INFINITY, mb = -INFINITY;
#pragma unroll
    for (int kt = 0; kt < 8; ++kt) {
      ma = fmaxf(ma, fmaxf(s[kt][0], s[kt][1]));
      mb = fmaxf(mb, fmaxf(s[kt][2], s[kt][3]));
    }
#pragma unroll
    for (int x = 1; x < 4; x <<= 1) {
      ma = fmaxf(ma, __shfl_xor_sync(0xffffffffu, ma, x));
      mb = fmaxf(mb, __shfl_xor_sync(0xffffffffu, mb, x));
    }
    ma = fmaxf(m_a, ma);  // finite from the first tile on, which holds key 0
    mb = fmaxf(m_b, mb);
    const float fa = ex2(m_a - ma), fb = ex2(m_b - mb);
    m_a = ma;
    m_b = mb;
    if (__any_sync(0xffffffffu, fa != 1.0f || fb != 1.0f)) {
      l_a *= fa;
      l_b *= fb;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        o[i][0] *= fa;
        o[i][1] *= fa;
        o[i][2] *= fb;
        o[i][3] *= fb;
      }
    }
    cp_async_wait<0>();
    __syncthreads();  // the values have landed; everybody is done with the keys
    if (t + 1 < tiles) {
      load_k(t + 1);
      cp_async_commit();
    }
#pragma unroll
    for (int kb = 0; kb < 4; ++kb) {
      uint32_t ph[4], pl[4];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const float* x = s[2 * kb + e];
        const float w0 = ex2(x[0] - ma), w1 = ex2(x[1] - ma);
        const float w2 = ex2(x[2] - mb), w3 = ex2(x[3] - mb);
        l_a += w0 + w1;
        l_b += w2 + w3;
        split2(w0, w1, ph[2 * e], pl[2 * e]);
        split2(w2, w3, ph[2 * e + 1], pl[2 * e + 1]);
      }
#pragma unroll
      for (int np = 0; np < NV / 2; np += 2) {  // four products between two that depend on one another
        if (16 * np >= dv) break;
        uint32_t v[2][4];
#pragma unroll
        for (int x = 0; x < 2; ++x) ldmatrix_x4_trans(v[x], v_a + uint32_t(kb * 16 * vs + (np + x) * 16) * 2);
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          mma_bf16_16816(o[2 * (np + x)], pl, v[x][0], v[x][1]);
          mma_bf16_16816(o[2 * (np + x) + 1], pl, v[x][2], v[x][3]);
        }
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          mma_bf16_16816(o[2 * (np + x)], ph, v[x][0], v[x][1]);
          mma_bf16_16816(o[2 * (np + x) + 1], ph, v[x][2], v[x][3]);
        }
      }
    }
    if (t + 1 < tiles) {
      cp_async_wait<0>();
      __syncthreads();  // the next keys have landed; everybody is done with the values
      load_v(t + 1);
      cp_async_commit();
    }
  }
#pragma unroll
  for (int x = 1; x < 4; x <<= 1) {
    l_a += __shfl_xor_sync(0xffffffffu, l_a, x);
    l_b += __shfl_xor_sync(0xffffffffu, l_b, x);
  }
  // whole pairs of numbers: every row and head starts at a multiple of four bytes
  const bool pairs = ((p.vdim | p.ld_out | (p.gate ? p.ld_gate : 0)) & 1) == 0 &&
                     ((reinterpret_cast<uintptr_t>(p.gate) | reinterpret_cast<uintptr_t>(p.out)) & 3) == 0;
#pragma unroll
  for (int hf = 0; hf < 2; ++hf) {
    const int r = ra + 8 * hf;
    if (r >= tokens) continue;
    const float inv = 1.0f / (hf ? l_b : l_a);
    const size_t row = size_t(start + i0 + r);
    const bf16* gate = p.gate ? static_cast<const bf16*>(p.gate) + row * p.ld_gate + (size_t)h * p.vdim : nullptr;
    bf16* out = static_cast<bf16*>(p.out) + row * p.ld_out + (size_t)h * p.vdim;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = 8 * i + 2 * t4;
      if (c >= p.vdim) continue;
      float y0 = o[i][2 * hf] * inv, y1 = o[i][2 * hf + 1] * inv;
      if (pairs) {
        if (gate) {
          const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gate + c));
          y0 *= sigmoid_f(x.x);
          y1 *= sigmoid_f(x.y);
        }
        *reinterpret_cast<__nv_bfloat162*>(out + c) = __floats2bfloat162_rn(y0, y1);
      } else {
        out[c] = __float2bfloat16_rn(gate ? y0 * sigmoid_f(__bfloat162float(gate[c])) : y0);
        if (c + 1 < p.vdim) out[c + 1] = __float2bfloat16_rn(gate ? y1 * sigmoid_f(__bfloat162float(gate[c + 1])) : y1);
      }
    }
  }
}

size_t smem_bytes(int dim, int vdim) {
  return size_t(kTile) * (size_t(2) * (up16(dim) + 8) + size_t(value_stride(vdim))) * 2;
}

template <int NV>
int launch(const q38_packed_attention_params& p, const q38_batch_desc& b, cudaStream_t s) {
  static const cudaError_t attr =
      cudaFuncSetAttribute(packed_attention_kernel<NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, max_optin_smem());
  Q38_CUDA_OK(attr);
  (void)launch_kernel(packed_attention_kernel<NV>, dim3(p.heads, (b.max_tokens_per_seq + kTile - 1) / kTile, b.num_seqs), dim3(kThreads),
                      smem_bytes(p.dim, p.vdim), s, p, b);
  Q38_LAUNCH_OK("packed_attention_kernel");
  return Q38_OK;
}

bool aligned16(const void* p, int ld) { return reinterpret_cast<uintptr_t>(p) % 16 == 0 && ld % 8 == 0; }

}  // namespace
}  // namespace q38

using namespace q38;

extern "C" int q38_packed_attention_fits(int dim, int vdim) {
  return dim > 0 && vdim > 0 && vdim <= 256 && dim <= 2048 && smem_bytes(dim, vdim) <= size_t(max_optin_smem());
}

extern "C" int q38_latent_gather(const q38_batch_desc* batch, const q38_kv_layer_desc* kv, int max_context, int rows, void* out,
                                 void* stream) {
  Q38_REQUIRE(batch && kv && out && kv->pages && kv->block_table, "latent_gather: null argument");
  Q38_REQUIRE(kv->dtype == Q38_KV_BF16 && kv->kv_heads == 1 && kv->v_dim == 0 && kv->k_dim % 32 == 0, "latent_gather: cache geometry");
  Q38_REQUIRE(batch->num_seqs > 0 && batch->num_seqs <= 65535 && max_context > 0 && rows > 0 && rows % kPage == 0, "latent_gather: sizes");
  Q38_REQUIRE(reinterpret_cast<uintptr_t>(out) % 16 == 0 && reinterpret_cast<uintptr_t>(kv->pages) % 16 == 0, "latent_gather: alignment");
  (void)launch_kernel(latent_gather_kernel, dim3((max_context + kPage - 1) / kPage, batch->num_seqs), dim3(256), 0, as_stream(stream), *batch,
                      *kv, rows, static_cast<bf16*>(out));
  Q38_LAUNCH_OK("latent_gather_kernel");
  return Q38_OK;
}

extern "C" int q38_packed_attention(const q38_packed_attention_params* p, const q38_batch_desc* batch, void* stream) {
  Q38_REQUIRE(p && batch && p->q && p->k && p->v && p->out, "packed_attention: null argument");
  if (batch->num_tokens == 0) return Q38_OK;
  Q38_REQUIRE(p->heads > 0 && p->heads <= 65535 && batch->num_seqs > 0 && batch->num_seqs <= 65535 && batch->max_tokens_per_seq > 0,
              "packed_attention: batch");
  Q38_REQUIRE(q38_packed_attention_fits(p->dim, p->vdim), "packed_attention: heads of %d / %d", p->dim, p->vdim);
  Q38_REQUIRE(p->q_stride >= up16(p->dim) && p->k_stride >= up16(p->dim) && p->v_stride >= up16(p->vdim) &&
                  (p->q_stride | p->k_stride | p->v_stride) % 8 == 0 && aligned16(p->q, p->ld_q) && aligned16(p->k, p->ld_kv) &&
                  aligned16(p->v, p->ld_kv), "packed_attention: heads must be padded to 16 numbers and start at multiples of 16 bytes");
  Q38_REQUIRE(p->ld_q >= p->heads * p->q_stride && p->ld_out >= p->heads * p->vdim && (!p->gate || p->ld_gate >= p->heads * p->vdim),
              "packed_attention: leading dimensions");
  const cudaStream_t s = as_stream(stream);
  if (p->vdim <= 64) return launch<8>(*p, *batch, s);
  if (p->vdim <= 128) return launch<16>(*p, *batch, s);
  return launch<32>(*p, *batch, s);
}
