// Attention with mixed heads on the tensor cores (mma.sync, bf16 operands, fp32 scores, weights and sums), for bf16 caches.
//
// A head's weights enter other heads' outputs, so they must be normalised before they are mixed, and a value product can
// only start once every head's weights of its keys are known. Both phases therefore come in two kernels:
//   decode   scores: one pass over K; the scores of a page go to a scratch indexed by the physical page ([page][head][64]),
//            each split of the keys leaves (maximum, sum). values: one pass over V; a warp normalises a page's scores with the
//            merged (maximum, sum), mixes the heads on the fly and multiplies. K and V are read once.
//   prefill  stats: (maximum, sum) per (token, head), flash-style without values. values: a CTA holds the heads' weights of
//            8 ... 64 tokens x 32 keys in shared memory, mixes them over the heads there, and every warp carries the output
//            of one (head, 128 value columns, 16 tokens) in registers.
// Operands of the decode kernels are loaded from global memory straight into fragments, those of prefill from staged tiles: 16
// contiguous bytes of a row (8 head dimensions of a key, or 8 keys of a value column - V is stored transposed) are the
// registers of two k16 steps under a permutation of k that both operands share.
#include <algorithm>
#include <type_traits>

#include "act.cuh"
#include "mixed_attention.h"

namespace q38 {
Q38_REGISTER_ERROR_WORD();
namespace {

using bf16 = __nv_bfloat16;
constexpr float kLog2e = 1.4426950408889634f;
constexpr int kPage = Q38_PAGE_TOKENS;

__device__ __forceinline__ const bf16* k_page(const q38_kv_layer_desc& kv, int page, int head) {
  return reinterpret_cast<const bf16*>(kv.pages + (size_t)page * kv.page_bytes) + (size_t)head * kPage * kv.k_dim;
}
__device__ __forceinline__ const bf16* v_page(const q38_kv_layer_desc& kv, int page, int head) {
  return reinterpret_cast<const bf16*>(kv.pages + (size_t)page * kv.page_bytes) + (size_t)kv.kv_heads * kPage * kv.k_dim +
         (size_t)head * kv.v_dim * kPage;
}
__device__ __forceinline__ uint4 ld16(const bf16* p) { return *reinterpret_cast<const uint4*>(p); }
__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// merge of two (maximum, sum) pairs in base 2
__device__ __forceinline__ void merge_ml(float& m, float& l, float m2, float l2) {
  const float nm = fmaxf(m, m2);
  l = (m == -INFINITY ? 0.0f : l * exp2f(m - nm)) + (m2 == -INFINITY ? 0.0f : l2 * exp2f(m2 - nm));
  m = nm;
}

// Row stride (elements) of a [rows][cols] bf16 tile in shared memory whose fragment reads (two rows x 64 bytes per
// phase) must not collide: an odd multiple of 64 bytes.
__host__ __device__ constexpr int tile_stride(int cols) { return cols % 64 == 32 ? cols : cols + 32; }

// ---- decode: scores -------------------------------------------------------------------------------------------------
constexpr int kDecWarps = 4;
struct SplitRange {
  int p0, p1, pages, active;  // this split's pages; pages of the sequence; splits that have any
};
__device__ __forceinline__ SplitRange split_range(int pos, int split, int splits) {
  const int pages = pos / kPage + 1, per = (pages + splits - 1) / splits;
  return {min(pages, split * per), min(pages, (split + 1) * per), pages, (pages + per - 1) / per};
}
// record of one (sequence, split, head): v_dim floats of output, then maximum and sum
__device__ __forceinline__ float* split_record(const q38_mixed_attention_params& p, const q38_kv_layer_desc& kv, int seq,
                                               int split, int splits, int h) {
  return p.partials + (((size_t)seq * splits + split) * p.heads + h) * (kv.v_dim + 2);
}

__global__ void __launch_bounds__(kDecWarps * 32)
mixed_decode_scores_kernel(q38_mixed_attention_params p, q38_batch_desc b, q38_kv_layer_desc kv, int splits) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ float red[kDecWarps][16][2];
  bf16* q_sm = reinterpret_cast<bf16*>(smem);  // [16][stride]
  const int qs = tile_stride(kv.k_dim), kb_n = kv.k_dim / 32;
  const int head = blockIdx.x, split = blockIdx.y, seq = blockIdx.z;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
  const int row = b.seq_start[seq], pos = b.tok_pos[seq], slot = b.seq_slot[seq];
  const int group = p.heads / kv.kv_heads;
  const SplitRange r = split_range(pos, split, splits);
  if (r.p0 >= r.p1) return;  // inactive splits are skipped by every reader
  const int* table = kv.block_table + (size_t)slot * kv.max_pages_per_seq;
  const float scale2 = p.scale * kLog2e;
  for (int h0 = 0; h0 < group; h0 += 16) {
    const int rows = min(16, group - h0);
    __syncthreads();
    const bf16* q = static_cast<const bf16*>(p.q) + ((size_t)row * p.heads + head * group + h0) * kv.k_dim;
    for (int i = threadIdx.x; i < 16 * kv.k_dim / 8; i += blockDim.x) {
      const int rr = i / (kv.k_dim / 8), c = i % (kv.k_dim / 8);
      *reinterpret_cast<uint4*>(q_sm + rr * qs + c * 8) = rr < rows ? ld16(q + (size_t)rr * kv.k_dim + c * 8) : make_uint4(0, 0, 0, 0);
    }
    __syncthreads();
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
    for (int pg = r.p0 + warp; pg < r.p1; pg += kDecWarps) {
      const int page = table[pg];
      const bf16* K = k_page(kv, page, head) + (size_t)g * kv.k_dim + t * 8;
      float acc[8][4] = {};
      for (int kb = 0; kb < kb_n; ++kb) {
        uint4 bf[8];
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) bf[nt] = ld16(K + (size_t)nt * 8 * kv.k_dim + kb * 32);
        const AFragPair a = a_fragments(ld16(q_sm + g * qs + kb * 32 + t * 8), ld16(q_sm + (g + 8) * qs + kb * 32 + t * 8));
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) mma_pair(acc[nt], a, bf[nt]);
      }
      float* out = p.scores + ((size_t)page * p.heads + head * group + h0) * kPage;
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        float mx = m[hf];
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) {
          const int key = pg * kPage + nt * 8 + 2 * t;
          float &s0 = acc[nt][2 * hf], &s1 = acc[nt][2 * hf + 1];
          s0 = key <= pos ? s0 * scale2 : -INFINITY;
          s1 = key + 1 <= pos ? s1 * scale2 : -INFINITY;
          mx = fmaxf(mx, fmaxf(s0, s1));
        }
        float sum = 0.0f;
        if (mx != -INFINITY) {
#pragma unroll
          for (int nt = 0; nt < 8; ++nt) sum += ex2(acc[nt][2 * hf] - mx) + ex2(acc[nt][2 * hf + 1] - mx);
          l[hf] = (m[hf] == -INFINITY ? 0.0f : l[hf] * ex2(m[hf] - mx)) + sum;
          m[hf] = mx;
        }
        const int rr = g + 8 * hf;
        if (rr < rows)
#pragma unroll
          for (int nt = 0; nt < 8; ++nt)
            *reinterpret_cast<float2*>(out + (size_t)rr * kPage + nt * 8 + 2 * t) = make_float2(acc[nt][2 * hf], acc[nt][2 * hf + 1]);
      }
    }
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
#pragma unroll
      for (int o = 1; o < 4; o <<= 1) {
        const float om = __shfl_xor_sync(0xffffffffu, m[hf], o), ol = __shfl_xor_sync(0xffffffffu, l[hf], o);
        merge_ml(m[hf], l[hf], om, ol);
      }
      if (t == 0) {
        red[warp][g + 8 * hf][0] = m[hf];
        red[warp][g + 8 * hf][1] = l[hf];
      }
    }
    __syncthreads();
    if (threadIdx.x < rows) {
      float M = red[0][threadIdx.x][0], L = red[0][threadIdx.x][1];
      for (int w = 1; w < kDecWarps; ++w) merge_ml(M, L, red[w][threadIdx.x][0], red[w][threadIdx.x][1]);
      float* rec = split_record(p, kv, seq, split, splits, head * group + h0 + threadIdx.x) + kv.v_dim;
      rec[0] = M;
      rec[1] = L;
    }
  }
}

// ---- decode: values ---------------------------------------------------------------------------------------------------
// VT value tiles of 8 columns per CTA (the head's columns are cut over blockIdx.x beyond 128), GROUP rounded up to a power
// of two.
template <int GROUP, int VT>
__global__ void __launch_bounds__(kDecWarps * 32)
mixed_decode_values_kernel(q38_mixed_attention_params p, q38_batch_desc b, q38_kv_layer_desc kv, int splits, int vchunks) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ __align__(16) uint8_t smem[];
  const int H = p.heads, group = H / kv.kv_heads;
  float* mx_sm = reinterpret_cast<float*>(smem);                             // [H]
  float* t_sm = mx_sm + H;                                                   // [H][GROUP]: head_mix[h][g] / L_g
  bf16* w_sm = reinterpret_cast<bf16*>(smem + ((size_t)(H + H * GROUP) * 4 + 15) / 16 * 16);  // [warps][16][96]
  float* red = reinterpret_cast<float*>(w_sm + kDecWarps * 16 * 96);         // [warps][GROUP][VT * 8]
  const int head = blockIdx.x / vchunks, v0 = blockIdx.x % vchunks * VT * 8, split = blockIdx.y, seq = blockIdx.z;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
  const int row = b.seq_start[seq], pos = b.tok_pos[seq], slot = b.seq_slot[seq];
  const SplitRange r = split_range(pos, split, splits);
  if (r.p0 >= r.p1) return;
  for (int h = threadIdx.x; h < H; h += blockDim.x) {
    float M = -INFINITY, L = 0.0f;
    for (int s = 0; s < r.active; ++s) {
      const float* rec = split_record(p, kv, seq, s, splits, h) + kv.v_dim;
      merge_ml(M, L, rec[0], rec[1]);
    }
    mx_sm[h] = M;
    for (int o = 0; o < GROUP; ++o) {
      const int ho = head * group + o;
      const float w = o >= group ? 0.0f : p.head_mix ? p.head_mix[(size_t)ho * H + h] : float(ho == h);
      t_sm[h * GROUP + o] = w / L;
    }
  }
  bf16* W = w_sm + warp * 16 * 96;  // rows beyond GROUP stay zero
  for (int i = lane; i < 16 * 96 / 2; i += 32) reinterpret_cast<uint32_t*>(W)[i] = 0u;
  __syncthreads();
  const int* table = kv.block_table + (size_t)slot * kv.max_pages_per_seq;
  const int nvt = min(VT, (kv.v_dim - v0) / 8);
  float acc[VT][4] = {};
  for (int pg = r.p0 + warp; pg < r.p1; pg += kDecWarps) {
    const int page = table[pg];
    const float2* S = reinterpret_cast<const float2*>(p.scores + (size_t)page * H * kPage) + lane;
    const bf16* V = v_page(kv, page, head) + (size_t)(v0 + g) * kPage + t * 8;
    uint4 bf[8];  // the first values travel while the weights are computed
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (i < nvt) bf[i] = ld16(V + (size_t)i * 8 * kPage);
    float2 w[GROUP] = {};
#pragma unroll 8
    for (int h = 0; h < H; ++h) {
      const float2 s = S[h * (kPage / 2)];
      const float mx = mx_sm[h], e0 = ex2(s.x - mx), e1 = ex2(s.y - mx);
#pragma unroll
      for (int o = 0; o < GROUP; ++o) {
        const float f = t_sm[h * GROUP + o];
        w[o].x += f * e0;
        w[o].y += f * e1;
      }
    }
#pragma unroll
    for (int o = 0; o < GROUP; ++o)
      *reinterpret_cast<__nv_bfloat162*>(W + o * 96 + 2 * lane) = __floats2bfloat162_rn(w[o].x, w[o].y);
    __syncwarp();
#pragma unroll
    for (int kb = 0; kb < 2; ++kb) {
      const AFragPair a = a_fragments(ld16(W + g * 96 + kb * 32 + t * 8), ld16(W + (g + 8) * 96 + kb * 32 + t * 8));
#pragma unroll
      for (int n0 = 0; n0 < VT; n0 += 8) {
        if (kb > 0 || n0 > 0)
#pragma unroll
          for (int i = 0; i < 8; ++i)
            if (n0 + i < nvt) bf[i] = ld16(V + (size_t)(n0 + i) * 8 * kPage + kb * 32);
#pragma unroll
        for (int i = 0; i < 8; ++i)
          if (n0 + i < nvt) mma_pair(acc[n0 + i], a, bf[i]);
      }
    }
    __syncwarp();
  }
#pragma unroll
  for (int nt = 0; nt < VT; ++nt)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int o = g + 8 * (e >> 1);
      if (o < GROUP) red[((size_t)warp * GROUP + o) * VT * 8 + nt * 8 + 2 * t + (e & 1)] = acc[nt][e];
    }
  __syncthreads();
  for (int i = threadIdx.x; i < group * nvt * 8; i += blockDim.x) {
    const int o = i / (nvt * 8), c = i % (nvt * 8), ho = head * group + o;
    float v = 0.0f;
    for (int w = 0; w < kDecWarps; ++w) v += red[((size_t)w * GROUP + o) * VT * 8 + c];
    if (splits > 1) split_record(p, kv, seq, split, splits, ho)[v0 + c] = v;
    else if (v0 + c < p.vdim) static_cast<bf16*>(p.out)[(size_t)row * p.ld_out + (size_t)ho * p.vdim + v0 + c] = __float2bfloat16_rn(v);
  }
}

// sum of the splits' outputs (their weights are normalised over all keys already)
__global__ void __launch_bounds__(256)
mixed_decode_merge_kernel(q38_mixed_attention_params p, q38_batch_desc b, q38_kv_layer_desc kv, int splits) {
  pdl_wait();
  pdl_launch_dependents();
  const int seq = blockIdx.y, row = b.seq_start[seq];
  const int active = split_range(b.tok_pos[seq], 0, splits).active;
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= p.heads * p.vdim) return;
  const int h = i / p.vdim, d = i % p.vdim;
  float v = 0.0f;
#pragma unroll 4
  for (int s = 0; s < active; ++s) v += split_record(p, kv, seq, s, splits, h)[d];
  static_cast<bf16*>(p.out)[(size_t)row * p.ld_out + i] = __float2bfloat16_rn(v);
}

// ---- prefill: (maximum, sum) per (token, head) -----------------------------------------------------------------------------
constexpr int kStatWarps = 4, kStatRows = 128;
template <int KB>
__global__ void __launch_bounds__(kStatWarps * 32)
mixed_prefill_stats_kernel(q38_mixed_attention_params p, q38_batch_desc b, q38_kv_layer_desc kv, int tile_tokens, int splits) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ __align__(16) uint8_t smem[];
  const int k_dim = KB ? KB * 32 : kv.k_dim, ks = tile_stride(k_dim), kb_n = k_dim / 32, chunks = k_dim / 8;
  bf16* q_sm = reinterpret_cast<bf16*>(smem);   // [128][ks]
  bf16* k_sm = q_sm + kStatRows * ks;           // [2][64][ks]
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
  const int head = blockIdx.y / splits, split = blockIdx.y % splits, seq = blockIdx.z;
  const int group = p.heads / kv.kv_heads;
  const int start = b.seq_start[seq], count = b.seq_start[seq + 1] - start, pos0 = b.seq_pos0[seq], slot = b.seq_slot[seq];
  const int t0 = (int(gridDim.x) - 1 - int(blockIdx.x)) * tile_tokens;  // the longest tiles first
  if (t0 >= count) return;
  const int tokens = min(tile_tokens, count - t0);
  const int last = pos0 + t0 + tokens - 1, pages = last / kPage + 1;
  const int per = (pages + splits - 1) / splits, p0 = min(pages, split * per), p1 = min(pages, p0 + per);
  const int* table = kv.block_table + (size_t)slot * kv.max_pages_per_seq;
  const int k_row = threadIdx.x >> 4, k_chunk = threadIdx.x & 15;  // half a warp per key row
  auto stage = [&](int pg) {
    const bf16* src = k_page(kv, table[pg], head) + (size_t)k_row * kv.k_dim;
    bf16* dst = k_sm + (((pg - p0) & 1) * kPage + k_row) * ks;
    for (int r = k_row; r < kPage; r += kStatWarps * 2, src += kStatWarps * 2 * kv.k_dim, dst += kStatWarps * 2 * ks)
      for (int c = k_chunk; c < chunks; c += 16) cp_async16(dst + c * 8, src + c * 8);
    cp_async_commit();
  };
  if (p0 < p1) stage(p0);
  for (int i = threadIdx.x; i < kStatRows * chunks; i += blockDim.x) {
    const int rr = i / chunks, c = i % chunks, tok = rr / group, h = head * group + rr % group;
    *reinterpret_cast<uint4*>(q_sm + rr * ks + c * 8) =
        tok < tokens ? ld16(static_cast<const bf16*>(p.q) + ((size_t)(start + t0 + tok) * p.heads + h) * kv.k_dim + c * 8)
                     : make_uint4(0, 0, 0, 0);
  }
  const float scale2 = p.scale * kLog2e;
  int limit[2][2];  // last visible position of this lane's rows
  float m[2][2], l[2][2];
#pragma unroll
  for (int mt = 0; mt < 2; ++mt)
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      limit[mt][hf] = pos0 + t0 + (warp * 32 + mt * 16 + hf * 8 + g) / group;
      m[mt][hf] = -INFINITY;
      l[mt][hf] = 0.0f;
    }
  for (int pg = p0; pg < p1; ++pg) {
    if (pg + 1 < p1) {
      stage(pg + 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const bf16* K = k_sm + ((pg - p0) & 1) * kPage * ks + g * ks + t * 8;
    const bf16* Q = q_sm + (warp * 32 + g) * ks + t * 8;
    float acc[2][8][4] = {};
#pragma unroll
    for (int kb = 0; kb < (KB ? KB : kb_n); ++kb) {
      const AFragPair a[2] = {a_fragments(ld16(Q + kb * 32), ld16(Q + 8 * ks + kb * 32)),
                              a_fragments(ld16(Q + 16 * ks + kb * 32), ld16(Q + 24 * ks + kb * 32))};
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) {
        const uint4 bf = ld16(K + nt * 8 * ks + kb * 32);
        mma_pair(acc[0][nt], a[0], bf);
        mma_pair(acc[1][nt], a[1], bf);
      }
    }
    const bool edge = (pg + 1) * kPage - 1 > pos0 + t0;
#pragma unroll
    for (int mt = 0; mt < 2; ++mt)
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        float mx = m[mt][hf];
#pragma unroll
        for (int nt = 0; nt < 8; ++nt)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            float& s = acc[mt][nt][2 * hf + e];
            s *= scale2;
          }
        if (edge) {
          const int lim = limit[mt][hf] - pg * kPage - 2 * t;
#pragma unroll
          for (int nt = 0; nt < 8; ++nt)
#pragma unroll
            for (int e = 0; e < 2; ++e)
              if (nt * 8 + e > lim) acc[mt][nt][2 * hf + e] = -INFINITY;
        }
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) mx = fmaxf(mx, fmaxf(acc[mt][nt][2 * hf], acc[mt][nt][2 * hf + 1]));
        if (mx == -INFINITY) continue;
        float sum = 0.0f;
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) sum += ex2(acc[mt][nt][2 * hf] - mx) + ex2(acc[mt][nt][2 * hf + 1] - mx);
        l[mt][hf] = (m[mt][hf] == -INFINITY ? 0.0f : l[mt][hf] * ex2(m[mt][hf] - mx)) + sum;
        m[mt][hf] = mx;
      }
    __syncthreads();
  }
#pragma unroll
  for (int mt = 0; mt < 2; ++mt)
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
#pragma unroll
      for (int o = 1; o < 4; o <<= 1) {
        const float om = __shfl_xor_sync(0xffffffffu, m[mt][hf], o), ol = __shfl_xor_sync(0xffffffffu, l[mt][hf], o);
        merge_ml(m[mt][hf], l[mt][hf], om, ol);
      }
      const int rr = warp * 32 + mt * 16 + hf * 8 + g, tok = rr / group;
      if (t == 0 && tok < tokens) {
        const size_t i = size_t(start - b.seq_start[0] + t0 + tok);
        *reinterpret_cast<float2*>(p.stats + (((size_t)split * b.num_tokens + i) * p.heads + head * group + rr % group) * 2) =
            make_float2(m[mt][hf], l[mt][hf]);
      }
    }
}

// ---- prefill: values, operands straight from global memory ------------------------------------------------------------------
// For shapes whose K and V tiles do not fit into shared memory (many kv heads).
// 16 warps; warp = (row group of 16 tokens, output head, chunk of 128 value columns). Keys in tiles of 32.
constexpr int kValWarps = 16, kKeys = 32, kPStride = 40;
struct ValGeom {
  int row_groups;   // RG: 16-token groups per CTA
  int vchunks;      // 128-column chunks of a value head
  int out_heads;    // output heads per CTA = 16 / (RG * vchunks)
  int q_in_smem;
};
__global__ void __launch_bounds__(kValWarps * 32, 1)
mixed_prefill_direct_kernel(q38_mixed_attention_params p, q38_batch_desc b, q38_kv_layer_desc kv, ValGeom geo, int splits) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ __align__(16) uint8_t smem[];
  const int H = p.heads, RG = geo.row_groups, TQ = 16 * RG, HO = geo.out_heads, group = H / kv.kv_heads;
  const int HP = (HO + 3) & ~3;
  const int qs = tile_stride(kv.k_dim), kb_n = kv.k_dim / 32;
  float* P = reinterpret_cast<float*>(smem);                  // [H][TQ][kPStride] normalised weights
  float* T = P + (size_t)H * TQ * kPStride;                   // [H in][HP] mixing matrix, transposed
  float2* ml = reinterpret_cast<float2*>(T + (size_t)H * HP); // [H][TQ] (maximum, 1 / sum)
  bf16* W = reinterpret_cast<bf16*>(ml + (size_t)H * TQ);     // [HO][TQ][32] mixed weights
  bf16* q_sm = W + (size_t)HO * TQ * kKeys;                   // [H][TQ][qs] (when it fits)
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
  const int seq = blockIdx.z, ho0 = blockIdx.y * HO;
  const int start = b.seq_start[seq], count = b.seq_start[seq + 1] - start, pos0 = b.seq_pos0[seq], slot = b.seq_slot[seq];
  const int t0 = (int(gridDim.x) - 1 - int(blockIdx.x)) * TQ;  // the longest tiles first
  if (t0 >= count) return;
  const int tokens = min(TQ, count - t0), last = pos0 + t0 + tokens - 1;
  const int* table = kv.block_table + (size_t)slot * kv.max_pages_per_seq;
  const bf16* qg = static_cast<const bf16*>(p.q) + (size_t)(start + t0) * H * kv.k_dim;
  const size_t i0 = size_t(start - b.seq_start[0] + t0);
  for (int e = threadIdx.x; e < H * TQ; e += blockDim.x) {
    const int h = e / TQ, i = e % TQ;
    float M = -INFINITY, L = 0.0f;
    if (i < tokens)
      for (int s = 0; s < splits; ++s) {
        const float2 v = *reinterpret_cast<const float2*>(p.stats + (((size_t)s * b.num_tokens + i0 + i) * H + h) * 2);
        merge_ml(M, L, v.x, v.y);
      }
    ml[e] = i < tokens ? make_float2(M, 1.0f / L) : make_float2(0.0f, 0.0f);
  }
  for (int e = threadIdx.x; e < H * HP; e += blockDim.x) {
    const int h = e / HP, ho = ho0 + e % HP;
    T[e] = ho >= H || e % HP >= HO ? 0.0f : p.head_mix ? p.head_mix[(size_t)ho * H + h] : float(ho == h);
  }
  if (geo.q_in_smem) {
    const int chunks = kv.k_dim / 8;
    for (int e = threadIdx.x; e < H * TQ * chunks; e += blockDim.x) {
      const int c = e % chunks, h = e / chunks % H, i = e / (chunks * H);
      *reinterpret_cast<uint4*>(q_sm + ((size_t)h * TQ + i) * qs + c * 8) =
          i < tokens ? ld16(qg + ((size_t)i * H + h) * kv.k_dim + c * 8) : make_uint4(0, 0, 0, 0);
    }
  }
  __syncthreads();
  const float scale2 = p.scale * kLog2e;
  // this warp's output
  const int rg = warp % RG, vc = warp / RG % geo.vchunks, ho = warp / (RG * geo.vchunks);
  const bool live = ho < HO && ho0 + ho < H;
  const int v0 = vc * 128, nvt = live ? min(16, (kv.v_dim - v0) / 8) : 0;
  float acc[16][4] = {};
  for (int j0 = 0; j0 <= last; j0 += kKeys) {
    const int page = table[j0 / kPage], in_page = j0 % kPage;
    // weights of every head
    for (int u = warp; u < H * RG; u += kValWarps) {
      const int h = u / RG, r = u % RG;
      const bf16* K = k_page(kv, page, h / group) + (size_t)(in_page + g) * kv.k_dim + t * 8;
      float s[4][4] = {};
      if (geo.q_in_smem) {
        const bf16* Q = q_sm + ((size_t)h * TQ + r * 16 + g) * qs + t * 8;
        for (int kb = 0; kb < kb_n; kb += 2) {
          const bool two = kb + 1 < kb_n;
          uint4 bf[2][4];
#pragma unroll
          for (int nt = 0; nt < 4; ++nt) bf[0][nt] = ld16(K + (size_t)nt * 8 * kv.k_dim + kb * 32);
          if (two)
#pragma unroll
            for (int nt = 0; nt < 4; ++nt) bf[1][nt] = ld16(K + (size_t)nt * 8 * kv.k_dim + kb * 32 + 32);
          {
            const AFragPair a = a_fragments(ld16(Q + kb * 32), ld16(Q + 8 * qs + kb * 32));
#pragma unroll
            for (int nt = 0; nt < 4; ++nt) mma_pair(s[nt], a, bf[0][nt]);
          }
          if (two) {
            const AFragPair a = a_fragments(ld16(Q + kb * 32 + 32), ld16(Q + 8 * qs + kb * 32 + 32));
#pragma unroll
            for (int nt = 0; nt < 4; ++nt) mma_pair(s[nt], a, bf[1][nt]);
          }
        }
      } else {
        const int ia = r * 16 + g;
        const bf16* Q = qg + ((size_t)ia * H + h) * kv.k_dim + t * 8;
        const uint4 zero = make_uint4(0, 0, 0, 0);
        for (int kb = 0; kb < kb_n; ++kb) {
          const AFragPair a = a_fragments(ia < tokens ? ld16(Q + kb * 32) : zero,
                                          ia + 8 < tokens ? ld16(Q + (size_t)8 * H * kv.k_dim + kb * 32) : zero);
#pragma unroll
          for (int nt = 0; nt < 4; ++nt) mma_pair(s[nt], a, ld16(K + (size_t)nt * 8 * kv.k_dim + kb * 32));
        }
      }
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const int i = r * 16 + hf * 8 + g, lim = pos0 + t0 + i;
        const float2 st = ml[h * TQ + i];
        float* out = P + ((size_t)h * TQ + i) * kPStride + 2 * t;
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
          const int j = j0 + nt * 8 + 2 * t;
          const float w0 = j <= lim ? exp2f(s[nt][2 * hf] * scale2 - st.x) * st.y : 0.0f;
          const float w1 = j + 1 <= lim ? exp2f(s[nt][2 * hf + 1] * scale2 - st.x) * st.y : 0.0f;
          *reinterpret_cast<float2*>(out + nt * 8) = make_float2(w0, w1);
        }
      }
    }
    __syncthreads();
    // mixing: a thread takes key `lane` of two token rows and a run of output heads
    {
      const int pairs = TQ / 2;                        // row pairs (i, i + TQ / 2)
      const int parts = max(1, kValWarps / pairs);     // output-head ranges, in steps of four heads
      const int step = (HP / 4 + parts - 1) / parts * 4;
      for (int e = warp; e < pairs * parts; e += kValWarps) {
        const int i = e % pairs, part = e / pairs;
        const float *pa = P + (size_t)i * kPStride + lane, *pb = pa + (size_t)pairs * kPStride;
        const int end = min(HP, (part + 1) * step);
        for (int o0 = part * step; o0 < end; o0 += 4) {
          float xa[4] = {}, xb[4] = {};
          const int n = min(4, HO - o0);
#pragma unroll 4
          for (int h = 0; h < H; ++h) {
            const float4 f = *reinterpret_cast<const float4*>(T + (size_t)h * HP + o0);
            const float wa = pa[(size_t)h * TQ * kPStride], wb = pb[(size_t)h * TQ * kPStride];
            xa[0] += f.x * wa, xa[1] += f.y * wa, xa[2] += f.z * wa, xa[3] += f.w * wa;
            xb[0] += f.x * wb, xb[1] += f.y * wb, xb[2] += f.z * wb, xb[3] += f.w * wb;
          }
#pragma unroll
          for (int q = 0; q < 4; ++q)
            if (q < n) {
              W[((size_t)(o0 + q) * TQ + i) * kKeys + lane] = __float2bfloat16_rn(xa[q]);
              W[((size_t)(o0 + q) * TQ + i + pairs) * kKeys + lane] = __float2bfloat16_rn(xb[q]);
            }
        }
      }
    }
    __syncthreads();
    if (live) {
      const bf16* w = W + ((size_t)ho * TQ + rg * 16 + g) * kKeys + t * 8;
      const AFragPair a = a_fragments(ld16(w), ld16(w + 8 * kKeys));
      const bf16* V = v_page(kv, page, (ho0 + ho) / group) + (size_t)(v0 + g) * kPage + in_page + t * 8;
#pragma unroll
      for (int n0 = 0; n0 < 16; n0 += 8) {
        uint4 bf[8];
#pragma unroll
        for (int i = 0; i < 8; ++i)
          if (n0 + i < nvt) bf[i] = ld16(V + (size_t)(n0 + i) * 8 * kPage);
#pragma unroll
        for (int i = 0; i < 8; ++i)
          if (n0 + i < nvt) mma_pair(acc[n0 + i], a, bf[i]);
      }
    }
  }
  if (!live) return;
#pragma unroll
  for (int hf = 0; hf < 2; ++hf) {
    const int i = rg * 16 + hf * 8 + g;
    if (i >= tokens) continue;
    bf16* out = static_cast<bf16*>(p.out) + (size_t)(start + t0 + i) * p.ld_out + (size_t)(ho0 + ho) * p.vdim;
#pragma unroll
    for (int nt = 0; nt < 16; ++nt) {
      const int d = v0 + nt * 8 + 2 * t;
      if (nt < nvt && d < p.vdim) out[d] = __float2bfloat16_rn(acc[nt][2 * hf]);
      if (nt < nvt && d + 1 < p.vdim) out[d + 1] = __float2bfloat16_rn(acc[nt][2 * hf + 1]);
    }
  }
}

// ---- prefill: values, operands staged in shared memory --------------------------------------------------------------------------
// The same division of labour (16 warps, keys in tiles of 32) with K and V tiles copied asynchronously: K of the next tile
// travels while the weights are mixed and the values multiplied, V of the next one while its scores are computed. The
// mixing runs on the tensor cores too: T [out heads x heads] against the weights [heads x (token, key)], both split into
// bf16 hi + lo (hi hi + hi lo + lo hi, fp32 sums); a weight is stored as one word (hi, lo). The CTAs of a cluster share
// one token tile and divide its keys; their outputs (weights are normalised over all keys) are summed through the
// cluster's shared memory in rank order.
struct TileGeom {
  int tokens;       // of a tile
  int row_groups, vchunks, out_heads, q_in_smem, heads_per_mma;
  int v_heads;      // kv heads whose values a CTA needs at most
  int head_words;   // P: words per head = 16 RG * kPStride + 4
  int out_stride;   // W: elements per output head = 16 RG * 32 + 8
  // byte offsets
  int k, v, p, w, t, ml, q, bytes;
};
__device__ __forceinline__ float4 ld_cluster_f32x4(uint32_t local_addr, uint32_t rank) {
  uint32_t remote;
  float4 v;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(local_addr), "r"(rank));
  asm volatile("ld.shared::cluster.v4.f32 {%0,%1,%2,%3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(remote) : "memory");
  return v;
}
__device__ __forceinline__ void cluster_barrier() {
  __syncwarp();
  asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ uint32_t split_word(float x) {
  const bf16 h = __float2bfloat16_rn(x), l = __float2bfloat16_rn(x - __bfloat162float(h));
  return uint32_t(__bfloat16_as_ushort(h)) | uint32_t(__bfloat16_as_ushort(l)) << 16;
}

// two values as (hi, lo) words
__device__ __forceinline__ uint2 split_words(float a, float b) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const uint32_t hw = *reinterpret_cast<const uint32_t*>(&h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - __uint_as_float(hw << 16), b - __uint_as_float(hw & 0xffff0000u));
  const uint32_t lw = *reinterpret_cast<const uint32_t*>(&l);
  return make_uint2(__byte_perm(hw, lw, 0x5410), __byte_perm(hw, lw, 0x7632));
}

constexpr int kMaxMixHeads = 256;
// KB = k_dim / 32 where it is known at compile time, else 0; VT = value tiles of a warp; QS = queries in shared memory.
// HP = heads in the 16 rows of an MMA: 1 = 16 tokens of a head; 2 = 8 tokens of two heads of one kv head (row g + 8 is
// the second head's token g), for models with more heads than a CTA could otherwise put out.
template <int KB, int VT, bool QS, int HP>
__global__ void __launch_bounds__(kValWarps * 32, 1)
mixed_prefill_values_kernel(q38_mixed_attention_params p, q38_batch_desc b, q38_kv_layer_desc kv, TileGeom geo, int splits, int cluster) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ uint8_t kv_of[kMaxMixHeads];  // kv head of a query head
  const int H = p.heads, G = kv.kv_heads, RG = HP == 2 ? 1 : geo.row_groups, TQ = HP == 2 ? 8 : 16 * RG, HO = geo.out_heads, group = H / G;
  const int k_dim = KB ? KB * 32 : kv.k_dim, qs = tile_stride(k_dim), kb_n = k_dim / 32, k_steps = (H + 15) / 16, m_tiles = (HO + 15) / 16;
  bf16* k_sm = reinterpret_cast<bf16*>(smem + geo.k);            // [G][32][qs]
  bf16* v_sm = reinterpret_cast<bf16*>(smem + geo.v);            // [v_heads][v_dim][32]
  uint32_t* P = reinterpret_cast<uint32_t*>(smem + geo.p);       // [H][TQ][kPStride] (+4 per head)
  bf16* W = reinterpret_cast<bf16*>(smem + geo.w);               // [HO][TQ][32] (+8 per head)
  uint4* T = reinterpret_cast<uint4*>(smem + geo.t);             // [m_tiles][k_steps][32 lanes][hi, lo] A fragments
  float2* ml = reinterpret_cast<float2*>(smem + geo.ml);         // [H][TQ] (maximum, 1 / sum)
  bf16* q_sm = reinterpret_cast<bf16*>(smem + geo.q);            // [H][TQ][qs] (when it fits)
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
  const int seq = blockIdx.z, ho0 = blockIdx.y * HO, rank = int(blockIdx.x) % cluster;
  const int start = b.seq_start[seq], count = b.seq_start[seq + 1] - start, pos0 = b.seq_pos0[seq], slot = b.seq_slot[seq];
  const int t0 = (int(gridDim.x) / cluster - 1 - int(blockIdx.x) / cluster) * TQ;  // the longest tiles first
  if (t0 >= count) return;  // the same for all CTAs of the cluster
  const int tokens = min(TQ, count - t0), last = pos0 + t0 + tokens - 1;
  const int* table = kv.block_table + (size_t)slot * kv.max_pages_per_seq;
  const int key_tiles = last / kKeys + 1, c0 = rank * key_tiles / cluster, c1 = (rank + 1) * key_tiles / cluster;
  const int gv0 = ho0 / group, gv1 = min(G, (ho0 + HO - 1) / group + 1);

  // half a warp per key row, one kv head per turn; V rows of 32 keys are four 16-byte pieces
  const int k_row = warp * 2 + (lane >> 4), k_chunk = lane & 15, k_chunks = k_dim / 8;
  auto copy_k = [&](int c) {
    const bf16* src = k_page(kv, table[c / 2], 0) + (size_t)((c % 2) * kKeys + k_row) * k_dim;
    bf16* dst = k_sm + k_row * qs;
    for (int hd = 0; hd < G; ++hd, src += (size_t)kPage * k_dim, dst += kKeys * qs)
      for (int ch = k_chunk; ch < k_chunks; ch += 16) cp_async16(dst + ch * 8, src + ch * 8);
    cp_async_commit();
  };
  auto copy_v = [&](int c) {
    const int rows = (gv1 - gv0) * kv.v_dim;  // consecutive heads' rows are consecutive in the page and here
    const bf16* src = v_page(kv, table[c / 2], gv0) + (size_t)(c % 2) * kKeys + (threadIdx.x & 3) * 8;
    for (int r = threadIdx.x >> 2; r < rows; r += kValWarps * 8) cp_async16(v_sm + r * kKeys + (threadIdx.x & 3) * 8, src + (size_t)r * kPage);
    cp_async_commit();
  };
  if (c0 < c1) copy_k(c0);
  const int rg_shift = RG == 4 ? 2 : RG == 2 ? 1 : 0;
  for (int h = threadIdx.x; h < H; h += blockDim.x) kv_of[h] = uint8_t(h / group);

  const bf16* qg = static_cast<const bf16*>(p.q) + (size_t)(start + t0) * H * k_dim;
  const size_t i0 = size_t(start - b.seq_start[0] + t0);
  for (int e = threadIdx.x; e < H * TQ; e += blockDim.x) {
    const int h = e % H, i = e / H;
    float M = -INFINITY, L = 0.0f;
    if (i < tokens)
      for (int s = 0; s < splits; ++s) {
        const float2 v = *reinterpret_cast<const float2*>(p.stats + (((size_t)s * b.num_tokens + i0 + i) * H + h) * 2);
        merge_ml(M, L, v.x, v.y);
      }
    ml[h * TQ + i] = i < tokens ? make_float2(M, 1.0f / L) : make_float2(INFINITY, 0.0f);  // rows without a token: weight 0
  }
  for (int e = threadIdx.x; e < m_tiles * k_steps * 32; e += blockDim.x) {
    const int ln = e % 32, k = e / 32 % k_steps, r = e / (32 * k_steps) * 16 + ln / 4, c = k * 16 + ln % 4 * 2;
    uint32_t hi[4], lo[4];
#pragma unroll
    for (int f = 0; f < 4; ++f) {  // rows r, r + 8 x columns c, c + 8
      uint32_t w[2];
#pragma unroll
      for (int d = 0; d < 2; ++d) {
        const int o = r + (f & 1) * 8, h = c + (f >> 1) * 8 + d, ho = ho0 + o;
        w[d] = split_word(o >= HO || ho >= H || h >= H ? 0.0f : p.head_mix ? p.head_mix[(size_t)ho * H + h] : float(ho == h));
      }
      hi[f] = __byte_perm(w[0], w[1], 0x5410);
      lo[f] = __byte_perm(w[0], w[1], 0x7632);
    }
    T[2 * e] = make_uint4(hi[0], hi[1], hi[2], hi[3]);
    T[2 * e + 1] = make_uint4(lo[0], lo[1], lo[2], lo[3]);
  }
  if (QS) {
    const int chunks = k_dim / 8;
    for (int e = threadIdx.x; e < H * TQ * chunks; e += blockDim.x) {
      const int c = e % chunks, h = e / chunks % H, i = e / (chunks * H);
      *reinterpret_cast<uint4*>(q_sm + ((size_t)h * TQ + i) * qs + c * 8) =
          i < tokens ? ld16(qg + ((size_t)i * H + h) * k_dim + c * 8) : make_uint4(0, 0, 0, 0);
    }
  }
  const float scale2 = p.scale * kLog2e;
  const int rg = warp % RG, vc = warp / RG % geo.vchunks, ho = warp / (RG * geo.vchunks) * HP;
  const bool live = ho < HO && ho0 + ho < H;
  const int v0 = vc * 128, nvt = live ? min(VT, (kv.v_dim - v0) / 8) : 0;
  const int v_row = live ? ((ho0 + ho) / group - gv0) * kv.v_dim + v0 : 0;
  float acc[VT][4] = {};
  for (int c = c0; c < c1; ++c) {
    const int j0 = c * kKeys;
    // the accumulators take half the registers: addresses are recomputed per tile, not kept (and spilled) across tiles
    int tid = int(threadIdx.x);
    asm volatile("" : "+r"(tid));
    const int lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    cp_async_wait<0>();
    __syncthreads();  // K of this tile is here; the previous tile's weights and values are done with
    copy_v(c);
    const bool edge = j0 + kKeys - 1 > pos0 + t0;  // some row of the tile ends inside these keys
    for (int u = warp; u < (HP == 2 ? H / 2 : H << rg_shift); u += kValWarps) {
      const int h = HP == 2 ? 2 * u : u >> rg_shift, r = u & (RG - 1);
      const bf16* K = k_sm + (kv_of[h] * kKeys + g) * qs + t * 8;
      float s[4][4] = {};
      // rows beyond the tile's tokens read the last one's query; their weights are zero
      const int ia = (HP == 2 ? 0 : r * 16) + g, ib = HP == 2 ? g : ia + 8, hb = HP == 2 ? h + 1 : h;
      const bf16* q0 = QS ? q_sm + (h * TQ + ia) * qs + t * 8 : qg + ((size_t)min(ia, tokens - 1) * H + h) * k_dim + t * 8;
      const bf16* q8 = QS ? q_sm + (hb * TQ + ib) * qs + t * 8 : qg + ((size_t)min(ib, tokens - 1) * H + hb) * k_dim + t * 8;
#pragma unroll
      for (int kb = 0; kb < (KB ? KB : kb_n); ++kb) {
        const AFragPair a = a_fragments(ld16(q0 + kb * 32), ld16(q8 + kb * 32));
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) mma_pair(s[nt], a, ld16(K + nt * 8 * qs + kb * 32));
        if (VT == 16) asm volatile("" ::: "memory");
      }
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const int i = hf ? ib : ia, hh = hf ? hb : h, lim = pos0 + t0 + i - j0 - 2 * t;
        const float2 st = ml[hh * TQ + i];
        uint32_t* out = P + hh * geo.head_words + i * kPStride + 2 * t;
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
          float w0 = ex2(fmaf(s[nt][2 * hf], scale2, -st.x)) * st.y, w1 = ex2(fmaf(s[nt][2 * hf + 1], scale2, -st.x)) * st.y;
          if (edge) {
            if (nt * 8 > lim) w0 = 0.0f;
            if (nt * 8 + 1 > lim) w1 = 0.0f;
          }
          *reinterpret_cast<uint2*>(out + nt * 8) = split_words(w0, w1);
        }
      }
    }
    __syncthreads();
    if (c + 1 < c1) copy_k(c + 1);
    else cp_async_commit();  // an empty group keeps the count below the same
    // mixing: a warp takes the 32 keys (four column tiles) of one token row per row group; columns of heads that do not
    // exist meet zeros of T, so any finite word serves
    for (int it = warp; it < TQ * m_tiles; it += kValWarps) {
      const int i = HP == 2 ? it & 7 : it, mt = HP == 2 ? it >> 3 : 0;
      const uint32_t* col = P + i * kPStride + g;
      float d[4][4] = {};
      for (int k = 0; k < k_steps; ++k) {
        const uint4* tf = T + 2 * ((mt * k_steps + k) * 32 + lane);
        const uint4 ah4 = tf[0], al4 = tf[1];
        const uint32_t ah[4] = {ah4.x, ah4.y, ah4.z, ah4.w}, al[4] = {al4.x, al4.y, al4.z, al4.w};
        const uint32_t* c0p[4];
#pragma unroll
        for (int f = 0; f < 4; ++f) c0p[f] = col + min(k * 16 + 2 * t + (f & 1) + (f >> 1) * 8, H - 1) * geo.head_words;
#pragma unroll
        for (int n = 0; n < 4; ++n) {
          const uint32_t w0 = c0p[0][n * 8], w1 = c0p[1][n * 8], w2 = c0p[2][n * 8], w3 = c0p[3][n * 8];
          const uint32_t bh0 = __byte_perm(w0, w1, 0x5410), bl0 = __byte_perm(w0, w1, 0x7632);
          const uint32_t bh1 = __byte_perm(w2, w3, 0x5410), bl1 = __byte_perm(w2, w3, 0x7632);
          mma_bf16_16816(d[n], ah, bh0, bh1);
          mma_bf16_16816(d[n], ah, bl0, bl1);
          mma_bf16_16816(d[n], al, bh0, bh1);
        }
      }
      const int o = mt * 16 + g;
      bf16* to = W + o * geo.out_stride + i * kKeys + 2 * t;
#pragma unroll
      for (int hf = 0; hf < 2; ++hf)
        if (o + 8 * hf < HO)
#pragma unroll
          for (int n = 0; n < 4; ++n)
            *reinterpret_cast<__nv_bfloat162*>(to + hf * 8 * geo.out_stride + n * 8) = __floats2bfloat162_rn(d[n][2 * hf], d[n][2 * hf + 1]);
    }
    cp_async_wait<1>();
    __syncthreads();  // V of this tile and the mixed weights are here
    if (live) {
      const bf16* V = v_sm + (v_row + g) * kKeys + t * 8;
      const bf16* w = W + (size_t)ho * geo.out_stride + (rg * 16 + g) * kKeys + t * 8;
      const AFragPair a = a_fragments(ld16(w), ld16(w + (HP == 2 ? geo.out_stride : 8 * kKeys)));
#pragma unroll
      for (int i = 0; i < VT; ++i) {  // tiles beyond the head are not stored
        mma_pair(acc[i], a, ld16(V + i * 8 * kKeys));
        if (i % 4 == 3) asm volatile("" ::: "memory");  // no more than four loads ahead: the accumulators hold half the registers
      }
    }
  }
  auto store = [&](int wp, int nt, int ln, float4 v) {  // the fragment of lane `ln` of warp `wp`, value tile nt
    const int r = wp % RG, vch = wp / RG % geo.vchunks, unit = wp / (RG * geo.vchunks), gg = ln >> 2, tt = ln & 3;
    const int d = vch * 128 + nt * 8 + 2 * tt;
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int i = HP == 2 ? gg : r * 16 + hf * 8 + gg, o = HP == 2 ? 2 * unit + hf : unit;
      if (i >= tokens || o >= HO || ho0 + o >= H) continue;
      bf16* out = static_cast<bf16*>(p.out) + (size_t)(start + t0 + i) * p.ld_out + (size_t)(ho0 + o) * p.vdim + d;
      if (d < p.vdim) out[0] = __float2bfloat16_rn(hf ? v.z : v.x);
      if (d + 1 < p.vdim) out[1] = __float2bfloat16_rn(hf ? v.w : v.y);
    }
  };
  if (cluster == 1) {
#pragma unroll
    for (int nt = 0; nt < VT; ++nt)
      if (nt < nvt) store(warp, nt, lane, make_float4(acc[nt][0], acc[nt][1], acc[nt][2], acc[nt][3]));
    return;
  }
  float4* red = reinterpret_cast<float4*>(smem);  // [16 warps][NR value tiles][32 lanes] of one round
  cp_async_wait<0>();
  auto join = [&](auto tiles_per_round) {
    constexpr int NR = decltype(tiles_per_round)::value;
#pragma unroll
    for (int q = 0; q < VT / NR; ++q) {
      if (q * NR * 8 >= kv.v_dim) break;  // uniform: no warp holds further columns
      __syncthreads();
      cluster_barrier();  // everyone is done with its tiles / with reading the previous round
#pragma unroll
      for (int i = 0; i < NR; ++i)
        red[(warp * NR + i) * 32 + lane] = make_float4(acc[NR * q + i][0], acc[NR * q + i][1], acc[NR * q + i][2], acc[NR * q + i][3]);
      __syncthreads();
      cluster_barrier();
      for (int e = rank * (kValWarps * 32) + threadIdx.x; e < kValWarps * NR * 32; e += cluster * kValWarps * 32) {
        float4 v = make_float4(0, 0, 0, 0);
#pragma unroll 4
        for (int r = 0; r < cluster; ++r) {
          const float4 x = ld_cluster_f32x4(smem_u32(red + e), uint32_t(r));
          v.x += x.x, v.y += x.y, v.z += x.z, v.w += x.w;
        }
        const int wp = e / (32 * NR), nt = NR * q + e / 32 % NR, vch = wp / RG % geo.vchunks;
        if (vch * 128 + nt * 8 < kv.v_dim) store(wp, nt, e % 32, v);
      }
    }
  };
  if (geo.bytes >= kValWarps * VT * 32 * 16) join(std::integral_constant<int, VT>{});
  else join(std::integral_constant<int, 4>{});
  __syncthreads();
  cluster_barrier();  // nobody leaves while its shared memory is being read
}

// ---- host -----------------------------------------------------------------------------------------------------------------------
size_t val_smem(const q38_mixed_attention_params& p, const q38_kv_layer_desc& kv, const ValGeom& g) {
  const size_t H = size_t(p.heads), TQ = 16 * size_t(g.row_groups), HO = size_t(g.out_heads);
  size_t n = H * TQ * kPStride * 4 + H * ((HO + 3) / 4 * 4) * 4 + H * TQ * 8 + HO * TQ * kKeys * 2;
  if (g.q_in_smem) n += H * TQ * size_t(tile_stride(kv.k_dim)) * 2;
  return n;
}
bool val_geom(const q38_mixed_attention_params& p, const q38_kv_layer_desc& kv, ValGeom* out) {
  ValGeom g{};
  g.vchunks = (kv.v_dim + 127) / 128;
  if (g.vchunks > kValWarps) return false;
  const size_t limit = size_t(max_optin_smem());
  for (int rg : {4, 2, 1}) {
    if (rg > 1 && rg * g.vchunks * p.heads > kValWarps) continue;  // few heads: more tokens per CTA instead
    g.row_groups = rg;
    g.out_heads = std::max(1, std::min(p.heads, kValWarps / (rg * g.vchunks)));
    for (int q : {1, 0}) {
      g.q_in_smem = q;
      if (val_smem(p, kv, g) <= limit) {
        *out = g;
        return true;
      }
    }
  }
  return false;
}

bool tile_geom(const q38_mixed_attention_params& p, const q38_kv_layer_desc& kv, TileGeom* out) {
  TileGeom g{};
  const int H = p.heads, group = H / kv.kv_heads;
  g.vchunks = (kv.v_dim + 127) / 128;
  if (g.vchunks > kValWarps || H > kMaxMixHeads) return false;
  for (int form : {8, 4, 2, 1}) {  // 8: two heads per MMA; 4, 2, 1: row groups
    const int rg = form == 8 ? 1 : form;
    g.heads_per_mma = form == 8 ? 2 : 1;
    if (form == 8 && (group % 2 != 0 || H * g.vchunks <= kValWarps)) continue;  // more heads than a CTA's warps, in pairs
    if (rg > 1 && rg * g.vchunks * H > kValWarps) continue;                     // few heads: more tokens per CTA instead
    g.row_groups = rg;
    g.out_heads = std::max(1, std::min(H, g.heads_per_mma * (kValWarps / (rg * g.vchunks))));
    const int HO = g.out_heads, TQ = form == 8 ? 8 : 16 * rg;
    g.tokens = TQ;
    // kv heads that HO consecutive query heads can touch (the runs start at multiples of HO)
    g.v_heads = std::min(kv.kv_heads, HO % group == 0 ? HO / group : group % HO == 0 ? 1 : (HO + group - 2) / group + 1);
    g.head_words = TQ * kPStride + 4;
    g.out_stride = TQ * kKeys + 8;
    for (int q : {1, 0}) {
      if (q && form == 8) continue;
      int at = 0;
      auto take = [&](int bytes) {
        const int here = at;
        at = (at + bytes + 127) / 128 * 128;
        return here;
      };
      g.k = take(kv.kv_heads * kKeys * tile_stride(kv.k_dim) * 2);
      g.v = take(g.v_heads * kv.v_dim * kKeys * 2);
      g.p = take(H * g.head_words * 4);
      g.w = take(g.out_heads * g.out_stride * 2);
      g.t = take((g.out_heads + 15) / 16 * ((H + 15) / 16) * 32 * 32);
      g.ml = take(H * TQ * 8);
      g.q_in_smem = q;
      g.q = take(q ? H * TQ * tile_stride(kv.k_dim) * 2 : 0);
      // the cluster's reduction reuses the space; value tiles are read in whole 128-column chunks
      g.bytes = std::max({at, kValWarps * 4 * 32 * 16, g.v + (g.v_heads * kv.v_dim + 128) * kKeys * 2});
      if (g.bytes <= max_optin_smem() - 1024) {
        *out = g;
        return true;
      }
    }
  }
  return false;
}

template <int KB, int VT, bool QS, int HP>
int launch_values_as(const q38_mixed_attention_params& p, const q38_batch_desc& b, const q38_kv_layer_desc& kv, const TileGeom& g,
                     int splits, cudaStream_t s) {
  static const cudaError_t attr = cudaFuncSetAttribute(mixed_prefill_values_kernel<KB, VT, QS, HP>,
                                                       cudaFuncAttributeMaxDynamicSharedMemorySize, max_optin_smem() - 1024);
  Q38_CUDA_OK(attr);
  const int q_tiles = (b.max_tokens_per_seq + g.tokens - 1) / g.tokens, hb = (p.heads + g.out_heads - 1) / g.out_heads;
  // CTAs per token tile by a cost in key tiles of a context of about 2,048 keys: the longest CTA, or the average load of
  // an SM where there are several waves; starting and joining a CTA costs about as much as five tiles.
  int cluster = 1;
  double best = 0.0;
  for (int c = 1; c <= 8; c *= 2) {
    const double ctas = double(q_tiles) * hb * b.num_seqs * c, longest = 64.0 / c + 5.0;
    const double cost = ctas <= num_sms() ? longest : std::max(longest, 1.15 * ctas * (48.0 / c + 5.0) / num_sms());
    if (c == 1 || cost < best) {
      best = cost;
      cluster = c;
    }
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(q_tiles * cluster, hb, b.num_seqs);
  cfg.blockDim = dim3(kValWarps * 32);
  cfg.dynamicSmemBytes = size_t(g.bytes);
  cfg.stream = s;
  cudaLaunchAttribute attrs[2];
  int n = 0;
  if (dependent_launch_allowed()) {
    attrs[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attrs[n++].val.programmaticStreamSerializationAllowed = 1;
  }
  if (cluster > 1) {
    attrs[n].id = cudaLaunchAttributeClusterDimension;
    attrs[n].val.clusterDim.x = unsigned(cluster);
    attrs[n].val.clusterDim.y = 1;
    attrs[n++].val.clusterDim.z = 1;
  }
  cfg.attrs = attrs;
  cfg.numAttrs = unsigned(n);
  Q38_CUDA_OK(cudaLaunchKernelEx(&cfg, mixed_prefill_values_kernel<KB, VT, QS, HP>, p, b, kv, g, splits, cluster));
  return Q38_OK;
}
template <int KB>
int launch_values(const q38_mixed_attention_params& p, const q38_batch_desc& b, const q38_kv_layer_desc& kv, const TileGeom& g,
                  int splits, cudaStream_t s) {
  if (kv.v_dim <= 64)
    return g.heads_per_mma == 2 ? launch_values_as<KB, 8, false, 2>(p, b, kv, g, splits, s)
           : g.q_in_smem        ? launch_values_as<KB, 8, true, 1>(p, b, kv, g, splits, s)
                                : launch_values_as<KB, 8, false, 1>(p, b, kv, g, splits, s);
  return g.heads_per_mma == 2 ? launch_values_as<KB, 16, false, 2>(p, b, kv, g, splits, s)
         : g.q_in_smem        ? launch_values_as<KB, 16, true, 1>(p, b, kv, g, splits, s)
                              : launch_values_as<KB, 16, false, 1>(p, b, kv, g, splits, s);
}

template <int GROUP, int VT>
int launch_decode_values(const q38_mixed_attention_params& p, const q38_batch_desc& b, const q38_kv_layer_desc& kv, int splits,
                         cudaStream_t s) {
  const int vchunks = (kv.v_dim + VT * 8 - 1) / (VT * 8);
  const size_t smem = ((size_t)(p.heads + p.heads * GROUP) * 4 + 15) / 16 * 16 + size_t(kDecWarps) * 16 * 96 * 2 +
                      size_t(kDecWarps) * GROUP * VT * 8 * 4;
  static const cudaError_t attr = cudaFuncSetAttribute(mixed_decode_values_kernel<GROUP, VT>,
                                                       cudaFuncAttributeMaxDynamicSharedMemorySize, max_optin_smem());
  Q38_CUDA_OK(attr);
  (void)launch_kernel(mixed_decode_values_kernel<GROUP, VT>, dim3(kv.kv_heads * vchunks, splits, b.num_seqs), dim3(kDecWarps * 32),
                      smem, s, p, b, kv, splits, vchunks);
  Q38_LAUNCH_OK("mixed_decode_values_kernel");
  return Q38_OK;
}
template <int GROUP>
int launch_decode_values_v(const q38_mixed_attention_params& p, const q38_batch_desc& b, const q38_kv_layer_desc& kv, int splits,
                           cudaStream_t s) {
  return kv.v_dim <= 64 ? launch_decode_values<GROUP, 8>(p, b, kv, splits, s) : launch_decode_values<GROUP, 16>(p, b, kv, splits, s);
}

}  // namespace

bool mixed_prefill_mma_fits(const q38_mixed_attention_params& p, const q38_kv_layer_desc& kv) {
  ValGeom g;
  TileGeom t;
  return p.heads / kv.kv_heads <= kStatRows && kv.k_dim <= 256 && (tile_geom(p, kv, &t) || val_geom(p, kv, &g));
}

int mixed_prefill_mma(const q38_mixed_attention_params& p, const q38_batch_desc& b, const q38_kv_layer_desc& kv, cudaStream_t s) {
  const int group = p.heads / kv.kv_heads, tile = kStatRows / group;
  const int tiles = (b.max_tokens_per_seq + tile - 1) / tile;
  // the keys of a tile are cut over several CTAs when the tiles alone leave most of the GPU idle
  const int ctas = tiles * kv.kv_heads * b.num_seqs;
  const int splits = std::max(1, std::min({p.stat_splits, 5 * num_sms() / ctas, 8}));
  const size_t smem = size_t(kStatRows + 2 * kPage) * size_t(tile_stride(kv.k_dim)) * 2;
  const auto stats = kv.k_dim == 64    ? &mixed_prefill_stats_kernel<2>
                     : kv.k_dim == 128 ? &mixed_prefill_stats_kernel<4>
                                       : &mixed_prefill_stats_kernel<0>;
  Q38_CUDA_OK(cudaFuncSetAttribute(stats, cudaFuncAttributeMaxDynamicSharedMemorySize, max_optin_smem()));
  (void)launch_kernel(stats, dim3(tiles, kv.kv_heads * splits, b.num_seqs), dim3(kStatWarps * 32), smem, s, p, b, kv, tile, splits);
  Q38_LAUNCH_OK("mixed_prefill_stats_kernel");
  TileGeom tg;
  if (tile_geom(p, kv, &tg)) {
    switch (kv.k_dim) {
      case 64: return launch_values<2>(p, b, kv, tg, splits, s);
      case 128: return launch_values<4>(p, b, kv, tg, splits, s);
      default: return launch_values<0>(p, b, kv, tg, splits, s);
    }
  }
  ValGeom g;
  Q38_REQUIRE(val_geom(p, kv, &g), "mixed_attention: shape does not fit");
  static const cudaError_t attr2 = cudaFuncSetAttribute(mixed_prefill_direct_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, max_optin_smem());
  Q38_CUDA_OK(attr2);
  const int TQ = 16 * g.row_groups;
  (void)launch_kernel(mixed_prefill_direct_kernel, dim3((b.max_tokens_per_seq + TQ - 1) / TQ, (p.heads + g.out_heads - 1) / g.out_heads, b.num_seqs),
                      dim3(kValWarps * 32), val_smem(p, kv, g), s, p, b, kv, g, splits);
  Q38_LAUNCH_OK("mixed_prefill_direct_kernel");
  return Q38_OK;
}

bool mixed_decode_mma_fits(const q38_mixed_attention_params& p, const q38_kv_layer_desc& kv) {
  const int group = p.heads / kv.kv_heads;
  return p.scores && p.partials && p.max_splits > 0 && group <= 16 && kv.k_dim <= 1024 && p.heads <= 512;
}

int mixed_decode_mma(const q38_mixed_attention_params& p, const q38_batch_desc& b, const q38_kv_layer_desc& kv, cudaStream_t s) {
  const int group = p.heads / kv.kv_heads;
  const int splits = std::max(1, std::min({p.max_splits, 4 * num_sms() / (b.num_seqs * kv.kv_heads), 64}));
  const size_t smem = size_t(16) * size_t(tile_stride(kv.k_dim)) * 2;
  (void)launch_kernel(mixed_decode_scores_kernel, dim3(kv.kv_heads, splits, b.num_seqs), dim3(kDecWarps * 32), smem, s, p, b, kv, splits);
  Q38_LAUNCH_OK("mixed_decode_scores_kernel");
  const int rc = group == 1  ? launch_decode_values_v<1>(p, b, kv, splits, s)
                 : group <= 2 ? launch_decode_values_v<2>(p, b, kv, splits, s)
                 : group <= 4 ? launch_decode_values_v<4>(p, b, kv, splits, s)
                 : group <= 8 ? launch_decode_values_v<8>(p, b, kv, splits, s)
                              : launch_decode_values_v<16>(p, b, kv, splits, s);
  if (rc || splits == 1) return rc;
  (void)launch_kernel(mixed_decode_merge_kernel, dim3((p.heads * p.vdim + 255) / 256, b.num_seqs), dim3(256), 0, s, p, b, kv, splits);
  Q38_LAUNCH_OK("mixed_decode_merge_kernel");
  return Q38_OK;
}

}  // namespace q38
