// Latent attention of the layer-list architectures: every head's queries, brought into the latent space beforehand, meet one
// cached latent per token, which is key and value at once.
//
// bf16 cache: one tensor-core kernel (mma.sync, fp32 scores, weights and sums) for prompts and decoding. The heads of a token
//   and the tokens of a run are the same thing to it - rows that share the keys: a CTA takes 16, 32 or 64 consecutive rows
//   (token, head) of a sequence and walks its pages, a page (64 latents) at a time, through a two-stage cp.async ring; the
//   tile serves the scores as it lies and the values transposed by ldmatrix. The softmax weights enter the second product as
//   bf16 hi + lo (16 mantissa bits). With few rows the pages are divided over CTAs and a second kernel joins the pieces.
// fp32 cache and outsized latents: a CTA per (token, head) on the CUDA cores.
#include <algorithm>

#include "act.cuh"
#include "host_util.h"

namespace q38 {
Q38_REGISTER_ERROR_WORD();
namespace {

using bf16 = __nv_bfloat16;
constexpr int kPage = Q38_PAGE_TOKENS;
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// ---- norms of both latents, append ----------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) latent_append_kernel(q38_latent_append_params p, q38_batch_desc b, q38_kv_layer_desc kv) {
  pdl_wait();
  pdl_launch_dependents();
  __shared__ float red[33];
  const int m = blockIdx.x, pos = b.tok_pos[m], slot = b.seq_slot[b.tok_seq[m]];
  const T* row = static_cast<const T*>(p.proj) + (size_t)m * p.ld_proj;
  const T* c = row + p.q_rank;
  float sq = 0.0f, sc = 0.0f;
  for (int i = threadIdx.x; i < p.q_rank; i += blockDim.x) {
    const float v = to_f32(row[i]);
    sq += v * v;
  }
  for (int i = threadIdx.x; i < p.kv_rank; i += blockDim.x) {
    const float v = to_f32(c[i]);
    sc += v * v;
  }
  const float rq = 1.0f / sqrtf(block_sum(sq, red) / float(p.q_rank) + p.eps);
  const float rc = 1.0f / sqrtf(block_sum(sc, red) / float(p.kv_rank) + p.eps);
  T* q = static_cast<T*>(p.q_out) + (size_t)m * p.ld_q;
  for (int i = threadIdx.x; i < p.q_rank; i += blockDim.x) q[i] = from_f32<T>(to_f32(row[i]) * rq * p.q_gain[i]);
  const int page = kv.block_table[(size_t)slot * kv.max_pages_per_seq + pos / kPage];
  if (page < 0 || page >= kv.num_pages) {
    report_error(0x901);
    return;
  }
  T* dst = reinterpret_cast<T*>(kv.pages + (size_t)page * kv.page_bytes) + (size_t)(pos % kPage) * kv.k_dim;
  for (int i = threadIdx.x; i < kv.k_dim; i += blockDim.x)
    dst[i] = from_f32<T>(i < p.kv_rank ? to_f32(c[i]) * rc * p.kv_gain[i] : 0.0f);
}

// ---- any size, any precision --------------------------------------------------------------------------------------------------
constexpr int kGenThreads = 128, kGenKeys = 128;
template <typename T>
__global__ void __launch_bounds__(kGenThreads) latent_general_kernel(q38_latent_attention_params p, q38_batch_desc b, q38_kv_layer_desc kv) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ __align__(16) float sm[];
  float* q_sm = sm;                // [k_dim]
  float* acc = sm + kv.k_dim;      // [k_dim]
  float* w_sm = acc + kv.k_dim;    // [keys]
  __shared__ float red[8];
  const int i = blockIdx.x, h = blockIdx.y, row = b.seq_start[0] + i, pos = b.tok_pos[i];
  const int slot = b.seq_slot[b.tok_seq[i] - b.tok_seq[0]], lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int* table = kv.block_table + (size_t)slot * kv.max_pages_per_seq;
  const T* q = static_cast<const T*>(p.q) + ((size_t)row * p.heads + h) * kv.k_dim;
  for (int d = threadIdx.x; d < kv.k_dim; d += kGenThreads) {
    q_sm[d] = to_f32(q[d]) * p.scale;
    acc[d] = 0.0f;
  }
  __syncthreads();
  float m = -INFINITY, l = 0.0f;
  for (int j0 = 0; j0 <= pos; j0 += kGenKeys) {
    const int j = j0 + threadIdx.x, n = min(kGenKeys, pos + 1 - j0);
    float s = -INFINITY;
    if (j <= pos) {
      const T* c = reinterpret_cast<const T*>(kv.pages + (size_t)table[j / kPage] * kv.page_bytes) + (size_t)(j % kPage) * kv.k_dim;
      s = 0.0f;
      for (int d = 0; d < kv.k_dim; ++d) s += q_sm[d] * to_f32(c[d]);
    }
    const float wm = warp_max(s);
    if (lane == 0) red[warp] = wm;
    __syncthreads();
    const float nm = fmaxf(m, fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3])));
    const float w = j <= pos ? expf(s - nm) : 0.0f, f = expf(m - nm);
    w_sm[threadIdx.x] = w;
    const float ws = warp_sum(w);
    if (lane == 0) red[4 + warp] = ws;
    __syncthreads();
    l = l * f + (red[4] + red[5]) + (red[6] + red[7]);
    m = nm;
    for (int d = threadIdx.x; d < kv.k_dim; d += kGenThreads) {
      float a = acc[d] * f;
      for (int k = 0; k < n; ++k) {
        const int key = j0 + k;
        a += w_sm[k] * to_f32(reinterpret_cast<const T*>(kv.pages + (size_t)table[key / kPage] * kv.page_bytes)[(size_t)(key % kPage) * kv.k_dim + d]);
      }
      acc[d] = a;
    }
    __syncthreads();
  }
  T* out = static_cast<T*>(p.out) + ((size_t)row * p.heads + h) * kv.k_dim;
  for (int d = threadIdx.x; d < kv.k_dim; d += kGenThreads) out[d] = from_f32<T>(acc[d] / l);
}

// ---- tensor cores ---------------------------------------------------------------------------------------------------------------
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

constexpr int kMmaThreads = 256, kPS = kPage + 8;
__host__ __device__ constexpr int row_stride(int k_dim) { return k_dim + 8; }  // an odd multiple of 16 bytes
struct MmaSmem {
  int q, c, p_hi, p_lo, total;
  __host__ __device__ MmaSmem(int rows, int k_dim) {
    q = 0;
    c = q + rows * row_stride(k_dim) * 2;
    p_hi = c + 2 * kPage * row_stride(k_dim) * 2;
    p_lo = p_hi + rows * kPS * 2;
    total = p_lo + rows * kPS * 2;
  }
};

// What a block of rows has to do: its rows of the sequence and its share of the pages.
struct Share {
  int first, rows;       // rows (token * heads + head) within the sequence's run
  int p0, p1, active;    // pages [p0, p1); shares of this block that have any
};
__device__ __forceinline__ Share share_of(int block, int block_rows, int count, int heads, int pos0, int split, int splits) {
  Share s;
  s.first = block * block_rows;
  s.rows = min(block_rows, count * heads - s.first);
  if (s.rows <= 0) return {s.first, 0, 0, 0, 0};
  const int pages = (pos0 + (s.first + s.rows - 1) / heads) / kPage + 1, per = (pages + splits - 1) / splits;
  s.p0 = min(pages, split * per);
  s.p1 = min(pages, s.p0 + per);
  s.active = (pages + per - 1) / per;
  return s;
}
// piece of a row: k_dim unnormalised outputs, maximum (base 2), sum
__device__ __forceinline__ float* piece(const q38_latent_attention_params& p, int k_dim, size_t block, int split, int splits, int block_rows, int r) {
  return p.partials + ((block * splits + split) * block_rows + r) * size_t(k_dim + 2);
}

// RG row groups of 16 x CG = 8 / RG warps side by side; a warp scores 64 / CG keys of a page and carries NT * 8 columns of
// the output (k_dim up to CG * NT * 8).
template <int RG, int NT>
__global__ void __launch_bounds__(kMmaThreads, 1)
latent_mma_kernel(q38_latent_attention_params p, q38_batch_desc b, q38_kv_layer_desc kv, int splits) {
  constexpr int CG = 8 / RG, ROWS = 16 * RG, KT = 8 / CG;  // KT: 8-key tiles of a warp's scores
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ float mx[ROWS][CG], sum[ROWS][CG];
  const int k_dim = kv.k_dim, rs = row_stride(k_dim);
  const MmaSmem L(ROWS, k_dim);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int rg = warp / CG, cg = warp % CG;
  const int split = blockIdx.y, seq = blockIdx.z;
  pdl_wait();
  pdl_launch_dependents();
  const int start = b.seq_start[seq], count = b.seq_start[seq + 1] - start, pos0 = b.seq_pos0[seq], H = p.heads;
  const Share sh = share_of(blockIdx.x, ROWS, count, H, pos0, split, splits);
  if (sh.p0 >= sh.p1) return;
  const int* table = kv.block_table + (size_t)b.seq_slot[seq] * kv.max_pages_per_seq;
  const int pieces = k_dim / 8;
  // 16-byte pieces of a page dealt to the threads in order: row and column of the first, steps to the next
  const int r0 = tid / pieces, k0 = tid - r0 * pieces, dr = kMmaThreads / pieces, dk = kMmaThreads - dr * pieces;

  auto load_page = [&](int pg) {
    int page = table[pg];
    if (page < 0 || page >= kv.num_pages) {
      if (tid == 0) report_error(0x902);
      page = 0;
    }
    const bf16* src = reinterpret_cast<const bf16*>(kv.pages + (size_t)page * kv.page_bytes);
    bf16* dst = reinterpret_cast<bf16*>(smem + L.c) + (size_t)(pg & 1) * kPage * rs;
    int r = r0, k = k0;
    uint32_t to = smem_u32(dst);
    for (int i = tid; i < kPage * pieces; i += kMmaThreads) {
      cp_async16(to + uint32_t(r * rs + 8 * k) * 2, src + (size_t)i * 8, true);
      r += dr;
      k += dk;
      if (k >= pieces) {
        k -= pieces;
        ++r;
      }
    }
    cp_async_commit();
  };
  const bf16* q = static_cast<const bf16*>(p.q) + ((size_t)start * H + sh.first) * k_dim;
  for (int i = tid; i < ROWS * pieces; i += kMmaThreads) {
    const int r = i / pieces, k = i - r * pieces;
    cp_async16(smem_u32(smem + L.q) + uint32_t(r * rs + 8 * k) * 2, r < sh.rows ? q + (size_t)i * 8 : q, r < sh.rows);
  }
  load_page(sh.p0);

  const int ra = 16 * rg + g, rb = ra + 8;
  const int pos_a = ra < sh.rows ? pos0 + (sh.first + ra) / H : -1, pos_b = rb < sh.rows ? pos0 + (sh.first + rb) / H : -1;
  const float scale2 = p.scale * kLog2e;
  float m_a = -INFINITY, m_b = -INFINITY, l_a = 0.0f, l_b = 0.0f;
  float o[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[i][e] = 0.0f;
  const uint32_t q_a = smem_u32(smem + L.q) + ((16 * rg + (lane & 15)) * rs + (lane >> 4) * 8) * 2;
  const uint32_t ph_a = smem_u32(smem + L.p_hi) + ((16 * rg + (lane & 15)) * kPS + (lane >> 4) * 8) * 2;
  const uint32_t pl_a = ph_a + uint32_t(L.p_lo - L.p_hi);
  const int c0 = cg * NT * 8;  // first output column of this warp

  for (int pg = sh.p0; pg < sh.p1; ++pg) {
    cp_async_wait<0>();
    __syncthreads();  // the page has landed; everybody is done with the one before
    if (pg + 1 < sh.p1) load_page(pg + 1);
    const uint32_t c_a = smem_u32(smem + L.c) + uint32_t((pg & 1) * kPage * rs) * 2;

    // ---- scores of this warp's keys ----
    float s[KT][4] = {};
    const int key0 = cg * KT * 8;
    if (KT == 1) {  // 8 keys: two k16 steps per load
      const uint32_t k_a = c_a + ((key0 + (lane & 7)) * rs + (lane >> 3) * 8) * 2;
      float s2[4] = {};
#pragma unroll 4
      for (int k = 0; k < k_dim; k += 32) {
        uint32_t kf[4], a0[4], a1[4];
        ldmatrix_x4(kf, k_a + k * 2);
        ldmatrix_x4(a0, q_a + k * 2);
        ldmatrix_x4(a1, q_a + k * 2 + 32);
        mma_bf16_16816(s[0], a0, kf[0], kf[1]);
        mma_bf16_16816(s2, a1, kf[2], kf[3]);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) s[0][e] += s2[e];
    } else {
      const uint32_t k_a = c_a + ((key0 + (lane & 7) + ((lane >> 4) << 3)) * rs + ((lane >> 3) & 1) * 8) * 2;
      float s2[KT][4] = {};  // every other step: shorter chains of dependent products
#pragma unroll 2
      for (int k = 0; k < k_dim; k += 32) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          uint32_t a[4];
          ldmatrix_x4(a, q_a + (k + 16 * e) * 2);
#pragma unroll
          for (int kp = 0; kp < KT / 2; ++kp) {
            uint32_t kf[4];
            ldmatrix_x4(kf, k_a + (kp * 16 * rs + k + 16 * e) * 2);
            mma_bf16_16816(e ? s2[2 * kp] : s[2 * kp], a, kf[0], kf[1]);
            mma_bf16_16816(e ? s2[2 * kp + 1] : s[2 * kp + 1], a, kf[2], kf[3]);
          }
        }
      }
#pragma unroll
      for (int kt = 0; kt < KT; ++kt)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[kt][e] += s2[kt][e];
    }
    float ma = -INFINITY, mb = -INFINITY;
#pragma unroll
    for (int kt = 0; kt < KT; ++kt)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int key = pg * kPage + key0 + 8 * kt + 2 * t4 + e;
        s[kt][e] = key <= pos_a ? s[kt][e] * scale2 : -INFINITY;
        s[kt][2 + e] = key <= pos_b ? s[kt][2 + e] * scale2 : -INFINITY;
        ma = fmaxf(ma, s[kt][e]);
        mb = fmaxf(mb, s[kt][2 + e]);
      }
#pragma unroll
    for (int x = 1; x < 4; x <<= 1) {
      ma = fmaxf(ma, __shfl_xor_sync(0xffffffffu, ma, x));
      mb = fmaxf(mb, __shfl_xor_sync(0xffffffffu, mb, x));
    }
    if (t4 == 0) {
      mx[ra][cg] = ma;
      mx[rb][cg] = mb;
    }
    __syncthreads();
#pragma unroll
    for (int x = 0; x < CG; ++x) {
      ma = fmaxf(ma, mx[ra][x]);
      mb = fmaxf(mb, mx[rb][x]);
    }
    ma = fmaxf(ma, m_a);
    mb = fmaxf(mb, m_b);
    const float base_a = ma == -INFINITY ? 0.0f : ma, base_b = mb == -INFINITY ? 0.0f : mb;
    const float fa = ex2(m_a - base_a), fb = ex2(m_b - base_b);
    m_a = ma;
    m_b = mb;
    l_a *= fa;
    l_b *= fb;
    // ---- weights: this warp's keys into shared memory, hi + lo ----
#pragma unroll
    for (int kt = 0; kt < KT; ++kt)
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const float base = hf ? base_b : base_a;
        const float w0 = ex2(s[kt][2 * hf] - base), w1 = ex2(s[kt][2 * hf + 1] - base);
        (hf ? l_b : l_a) += w0 + w1;
        const __nv_bfloat162 hi = __floats2bfloat162_rn(w0, w1);
        const float2 f = __bfloat1622float2(hi);
        const int at = ((hf ? rb : ra) * kPS + key0 + 8 * kt + 2 * t4) * 2;
        *reinterpret_cast<__nv_bfloat162*>(smem + L.p_hi + at) = hi;
        *reinterpret_cast<__nv_bfloat162*>(smem + L.p_lo + at) = __floats2bfloat162_rn(w0 - f.x, w1 - f.y);
      }
    if (__any_sync(0xffffffffu, fa != 1.0f || fb != 1.0f)) {
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        o[i][0] *= fa;
        o[i][1] *= fa;
        o[i][2] *= fb;
        o[i][3] *= fb;
      }
    }
    __syncthreads();
    // ---- outputs: all keys of the page, this warp's columns ----
    const uint32_t v_a = c_a + (((lane & 7) + (((lane >> 3) & 1) << 3)) * rs + c0 + (lane >> 4) * 8) * 2;
#pragma unroll
    for (int kb = 0; kb < kPage / 16; ++kb) {
      uint32_t ph[4], pl[4];
      ldmatrix_x4(ph, ph_a + kb * 32);
      ldmatrix_x4(pl, pl_a + kb * 32);
#pragma unroll
      for (int np = 0; np < NT / 2; ++np) {
        if (c0 + 16 * np >= k_dim) break;
        uint32_t v[4];
        ldmatrix_x4_trans(v, v_a + (kb * 16 * rs + np * 16) * 2);
        mma_bf16_16816(o[2 * np], pl, v[0], v[1]);
        mma_bf16_16816(o[2 * np + 1], pl, v[2], v[3]);
        mma_bf16_16816(o[2 * np], ph, v[0], v[1]);
        mma_bf16_16816(o[2 * np + 1], ph, v[2], v[3]);
      }
    }
  }
  // ---- the rows' sums over all warps ----
#pragma unroll
  for (int x = 1; x < 4; x <<= 1) {
    l_a += __shfl_xor_sync(0xffffffffu, l_a, x);
    l_b += __shfl_xor_sync(0xffffffffu, l_b, x);
  }
  if (t4 == 0) {
    sum[ra][cg] = l_a;
    sum[rb][cg] = l_b;
  }
  __syncthreads();
  l_a = l_b = 0.0f;
#pragma unroll
  for (int x = 0; x < CG; ++x) {
    l_a += sum[ra][x];
    l_b += sum[rb][x];
  }
#pragma unroll
  for (int hf = 0; hf < 2; ++hf) {
    const int r = hf ? rb : ra;
    if (r >= sh.rows) continue;
    if (splits == 1) {
      const float inv = 1.0f / (hf ? l_b : l_a);
      bf16* out = static_cast<bf16*>(p.out) + ((size_t)start * H + sh.first + r) * k_dim + c0 + 2 * t4;
#pragma unroll
      for (int i = 0; i < NT; ++i)
        if (c0 + 8 * i < k_dim)
          *reinterpret_cast<__nv_bfloat162*>(out + 8 * i) = __floats2bfloat162_rn(o[i][2 * hf] * inv, o[i][2 * hf + 1] * inv);
    } else {
      float* rec = piece(p, k_dim, (size_t)seq * gridDim.x + blockIdx.x, split, splits, ROWS, r);
#pragma unroll
      for (int i = 0; i < NT; ++i)
        if (c0 + 8 * i < k_dim) *reinterpret_cast<float2*>(rec + c0 + 8 * i + 2 * t4) = make_float2(o[i][2 * hf], o[i][2 * hf + 1]);
      if (cg == 0 && t4 == 0) *reinterpret_cast<float2*>(rec + k_dim) = make_float2(hf ? m_b : m_a, hf ? l_b : l_a);
    }
  }
}

// Joins the pieces of a row; one CTA per row.
__global__ void __launch_bounds__(128) latent_join_kernel(q38_latent_attention_params p, q38_batch_desc b, int k_dim, int blocks, int block_rows, int splits) {
  pdl_wait();
  pdl_launch_dependents();
  __shared__ float factor[64];
  const int seq = blockIdx.y, row = blockIdx.x, block = row / block_rows, r = row % block_rows;
  const int start = b.seq_start[seq], count = b.seq_start[seq + 1] - start;
  const Share sh = share_of(block, block_rows, count, p.heads, b.seq_pos0[seq], 0, splits);
  if (r >= sh.rows) return;
  const size_t at = (size_t)seq * blocks + block;
  if (threadIdx.x < 32) {
    float m[2], l[2], top = -INFINITY, total = 0.0f;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int s = threadIdx.x + 32 * e;
      m[e] = -INFINITY;
      l[e] = 0.0f;
      if (s < sh.active) {
        const float2 ml = *reinterpret_cast<const float2*>(piece(p, k_dim, at, s, splits, block_rows, r) + k_dim);
        m[e] = ml.x;
        l[e] = ml.y;
      }
      top = fmaxf(top, m[e]);
    }
    top = warp_max(top);
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      m[e] = m[e] == -INFINITY ? 0.0f : ex2(m[e] - top);
      total += m[e] * l[e];
    }
    total = warp_sum(total);
    factor[threadIdx.x] = m[0] / total;
    factor[threadIdx.x + 32] = m[1] / total;
  }
  __syncthreads();
  bf16* out = static_cast<bf16*>(p.out) + ((size_t)start * p.heads + row) * k_dim;
  for (int c = 2 * threadIdx.x; c < k_dim; c += 256) {
    float2 v = make_float2(0, 0);
    for (int s = 0; s < sh.active; ++s) {
      const float2 x = *reinterpret_cast<const float2*>(piece(p, k_dim, at, s, splits, block_rows, r) + c);
      v.x += factor[s] * x.x;
      v.y += factor[s] * x.y;
    }
    *reinterpret_cast<__nv_bfloat162*>(out + c) = __floats2bfloat162_rn(v.x, v.y);
  }
}

constexpr int kMaxKDim = 512, kMaxSplits = 64;
constexpr int kPieceRows = 64;  // rows of pieces per SM that the scratch holds: 64-row CTAs one per SM, 16-row CTAs four

template <int RG, int NT>
int launch_mma(const q38_latent_attention_params& p, const q38_batch_desc& b, const q38_kv_layer_desc& kv, cudaStream_t s) {
  constexpr int ROWS = 16 * RG;
  const MmaSmem L(ROWS, kv.k_dim);
  static const cudaError_t attr =
      cudaFuncSetAttribute(latent_mma_kernel<RG, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, max_optin_smem() - 1024);
  Q38_CUDA_OK(attr);
  const int blocks = (b.max_tokens_per_seq * p.heads + ROWS - 1) / ROWS;
  const long long ctas = (long long)blocks * b.num_seqs;
  // Few CTAs: the pages of each over as many as there is room for (and scratch for the pieces).
  const int resident = std::min(4 / RG, std::max(1, 220 * 1024 / (L.total + 1024 + 2 * ROWS * 8 * 4)));
  int splits = int(std::min<long long>(kMaxSplits, (long long)num_sms() * resident / ctas));
  const size_t per_split = size_t(ctas) * ROWS * size_t(kv.k_dim + 2);
  if (!p.partials) splits = 1;
  else splits = std::max(1, std::min(splits, int(std::min<size_t>(kMaxSplits, p.partial_floats / per_split))));
  (void)launch_kernel(latent_mma_kernel<RG, NT>, dim3(blocks, splits, b.num_seqs), dim3(kMmaThreads), size_t(L.total), s, p, b, kv, splits);
  Q38_LAUNCH_OK("latent_mma_kernel");
  if (splits > 1) {
    (void)launch_kernel(latent_join_kernel, dim3(b.max_tokens_per_seq * p.heads, b.num_seqs), dim3(128), 0, s, p, b, kv.k_dim, blocks, ROWS, splits);
    Q38_LAUNCH_OK("latent_join_kernel");
  }
  return Q38_OK;
}

template <int RG>
int launch_rows(const q38_latent_attention_params& p, const q38_batch_desc& b, const q38_kv_layer_desc& kv, cudaStream_t s) {
  constexpr int CG = 8 / RG;
  if (kv.k_dim <= 128) return launch_mma<RG, 16 / CG>(p, b, kv, s);
  if (kv.k_dim <= 256) return launch_mma<RG, 32 / CG>(p, b, kv, s);
  return launch_mma<RG, 64 / CG>(p, b, kv, s);
}

template <typename T>
int launch_general(const q38_latent_attention_params& p, const q38_batch_desc& b, const q38_kv_layer_desc& kv, cudaStream_t s) {
  const size_t smem = (size_t(2) * kv.k_dim + kGenKeys) * 4;
  Q38_REQUIRE(smem <= size_t(max_optin_smem() - 1024), "latent_attention: latents of %d do not fit", kv.k_dim);
  static const cudaError_t attr =
      cudaFuncSetAttribute(latent_general_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, max_optin_smem() - 1024);
  Q38_CUDA_OK(attr);
  (void)launch_kernel(latent_general_kernel<T>, dim3(b.num_tokens, p.heads), dim3(kGenThreads), smem, s, p, b, kv);
  Q38_LAUNCH_OK("latent_general_kernel");
  return Q38_OK;
}

int check_cache(const char* what, const q38_batch_desc* b, const q38_kv_layer_desc* kv, int act) {
  Q38_REQUIRE(b->seq_start && b->seq_slot && b->seq_pos0 && b->tok_pos && b->tok_seq && b->num_seqs > 0 && b->num_seqs <= 65535 &&
                  b->max_tokens_per_seq > 0, "%s: batch", what);
  Q38_REQUIRE(kv->pages && kv->block_table && kv->kv_heads == 1 && kv->v_dim == 0 && kv->k_dim > 0 && kv->k_dim % 32 == 0, "%s: cache geometry", what);
  Q38_REQUIRE(act == Q38_ACT_BF16 || act == Q38_ACT_F32, "%s: activation precision %d", what, act);
  Q38_REQUIRE(kv->dtype == (act == Q38_ACT_BF16 ? Q38_KV_BF16 : Q38_KV_F32), "%s: cache precision %d", what, kv->dtype);
  return Q38_OK;
}

}  // namespace
}  // namespace q38

using namespace q38;

extern "C" int q38_latent_append(const q38_latent_append_params* p, const q38_batch_desc* batch, const q38_kv_layer_desc* kv,
                                 void* stream) {
  Q38_REQUIRE(p && batch && kv && p->proj && p->q_gain && p->kv_gain && p->q_out, "latent_append: null argument");
  if (batch->num_tokens == 0) return Q38_OK;
  if (const int rc = check_cache("latent_append", batch, kv, p->act)) return rc;
  Q38_REQUIRE(p->q_rank > 0 && p->kv_rank > 0 && p->kv_rank <= kv->k_dim && p->ld_proj >= p->q_rank + p->kv_rank && p->ld_q >= p->q_rank,
              "latent_append: ranks %d, %d", p->q_rank, p->kv_rank);
  if (p->act == Q38_ACT_BF16)
    (void)launch_kernel(latent_append_kernel<bf16>, dim3(batch->num_tokens), dim3(256), 0, as_stream(stream), *p, *batch, *kv);
  else
    (void)launch_kernel(latent_append_kernel<float>, dim3(batch->num_tokens), dim3(256), 0, as_stream(stream), *p, *batch, *kv);
  Q38_LAUNCH_OK("latent_append_kernel");
  return Q38_OK;
}

extern "C" size_t q38_latent_attention_partial_floats(int k_dim) {
  return size_t(num_sms()) * kPieceRows * size_t(k_dim + 2);
}

extern "C" int q38_latent_attention(const q38_latent_attention_params* p, const q38_batch_desc* batch, const q38_kv_layer_desc* kv,
                                    void* stream) {
  Q38_REQUIRE(p && batch && kv && p->q && p->out, "latent_attention: null argument");
  if (batch->num_tokens == 0) return Q38_OK;
  if (const int rc = check_cache("latent_attention", batch, kv, p->act)) return rc;
  Q38_REQUIRE(p->heads > 0 && p->heads <= 65535, "latent_attention: %d heads", p->heads);
  const cudaStream_t s = as_stream(stream);
  if (p->act == Q38_ACT_F32) return launch_general<float>(*p, *batch, *kv, s);
  if (kv->k_dim > kMaxKDim || (reinterpret_cast<uintptr_t>(p->q) | reinterpret_cast<uintptr_t>(p->out) | reinterpret_cast<uintptr_t>(kv->pages)) % 16 ||
      kv->page_bytes % 16)
    return launch_general<bf16>(*p, *batch, *kv, s);
  const int rows = batch->max_tokens_per_seq * p->heads;
  if (rows <= 16) return launch_rows<1>(*p, *batch, *kv, s);
  if (rows <= 32) return launch_rows<2>(*p, *batch, *kv, s);
  return launch_rows<4>(*p, *batch, *kv, s);
}
