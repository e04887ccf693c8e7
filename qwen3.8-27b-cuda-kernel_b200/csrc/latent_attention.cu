// Latent attention of the layer-list architectures: every head's queries, brought into the latent space beforehand, meet one
// cached latent per token, which is key and value at once.
//
// bf16 cache: tensor-core kernels (mma.sync, fp32 scores, weights and sums) for prompts and decoding. The heads of a token and
//   the tokens of a run are the same thing to them - rows that share the keys: a CTA takes 16, 32 or 64 consecutive rows
//   (token, head) of a sequence and walks its pages, 64 latents at a time, through a ring of TMA loads; a page serves the
//   scores as it lies and the values transposed by ldmatrix. What bounds this is the traffic between shared memory and the
//   fragments, so up to 32 rows keep their queries in registers: the warps divide the latent's dimensions (and the keys)
//   among them and add their parts of the scores through shared memory. The softmax weights enter the second product as
//   bf16 hi + lo (16 mantissa bits). With few rows the pages are divided over CTAs and a second kernel joins the pieces.
// fp32 cache and outsized latents: a CTA per (token, head) on the CUDA cores.
#include <algorithm>

#include "act.cuh"
#include "host_util.h"
#include "tensor_map.h"

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
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}

constexpr int kPS = kPage + 8;
__host__ __device__ constexpr int row_stride(int k_dim) { return k_dim + 8; }  // an odd multiple of 16 bytes
// A page in shared memory: tiles of 64 dimensions, [tile][64 latents][128 bytes] with the 128-byte swizzle, so that the eight
// rows of an ldmatrix phase lie in different banks.
constexpr int kTileBytes = kPage * 128;
__host__ __device__ constexpr int page_smem(int k_dim) { return (k_dim + 63) / 64 * kTileBytes; }
// byte offset of the 16 bytes at dimension 8 * chunk of latent `row` (the swizzle only depends on row & 7)
__device__ __forceinline__ uint32_t page_at(int row, int chunk) {
  return uint32_t((chunk >> 3) * kTileBytes + row * 128 + (((chunk & 7) ^ (row & 7)) << 4));
}

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

// The ring of pages of one CTA. Thread 0 asks for the pages, every thread sees every one of them, so one barrier per stage is
// enough. A wait that runs out makes the results meaningless; the kernel then asks for nothing more and drains.
template <int STAGES>
struct PageRing {
  uint64_t* full;  // [STAGES]
  int* issued;     // [STAGES] loads each barrier has been told about
  uint8_t* pages;  // 1024-byte aligned
  const int* table;
  int k_dim, first, last;

  // thread 0
  __device__ __forceinline__ void start(const CUtensorMap* map, int num_pages) const {
    for (int i = 0; i < STAGES; ++i) {
      mbar_init(&full[i], 1);
      issued[i] = 0;
    }
    mbar_fence_init();
    for (int i = 0; i < STAGES && first + i < last; ++i) load(map, num_pages, first + i);
  }
  __device__ __forceinline__ void load(const CUtensorMap* map, int num_pages, int pg) const {
    const int stage = (pg - first) % STAGES;
    int page = table[pg];
    if (page < 0 || page >= num_pages) {
      report_error(0x902);
      page = 0;
    }
    uint8_t* dst = pages + stage * page_smem(k_dim);
    mbar_expect_tx(&full[stage], uint32_t(page_smem(k_dim)));
    issued[stage] += 1;
    for (int d = 0; d < k_dim; d += 64) tma_load_2d(dst + d / 64 * kTileBytes, map, d, page * kPage, &full[stage]);
  }
  __device__ __forceinline__ bool wait(int pg) const {  // a whole warp, the same answer in all its lanes
    return __all_sync(0xffffffffu, mbar_wait(&full[(pg - first) % STAGES], uint32_t((pg - first) / STAGES) & 1, 0x904));
  }
  __device__ __forceinline__ uint32_t at(int pg) const { return smem_u32(pages) + uint32_t((pg - first) % STAGES * page_smem(k_dim)); }
  __device__ __forceinline__ void finish(bool ok) const {  // every thread; also a barrier
    if (__syncthreads_or(!ok) && threadIdx.x < STAGES && issued[threadIdx.x] > 0)
      for (uint32_t i = 0; i < kSpinLimit; ++i)
        if (mbar_try_wait(&full[threadIdx.x], uint32_t(issued[threadIdx.x] - 1) & 1)) break;
  }
};
__device__ __forceinline__ uint8_t* ring_base(uint8_t* smem) { return smem + ((1024 - (smem_u32(smem) & 1023)) & 1023); }

// Output column pair of a finished row: as it is stored, or into the row's piece.
struct RowOut {
  bf16* out;
  float* rec;
  float inv;
  __device__ __forceinline__ void put(int c, float a, float b) const {
    if (rec) *reinterpret_cast<float2*>(rec + c) = make_float2(a, b);
    else *reinterpret_cast<__nv_bfloat162*>(out + c) = __floats2bfloat162_rn(a * inv, b * inv);
  }
};

// Up to 32 rows (RG groups of 16). Scores: a warp takes a quarter of the dimensions (KS k16 steps, queries in registers) of
// 256 / WARPS keys; softmax: all threads, a row by neighbouring ones; outputs: a warp takes NT * 8 columns for all rows.
constexpr int kXS = kPage + 8;  // row stride of the parts of the scores, in floats
template <int RG, int WARPS, int KS, int NT, int STAGES>
__global__ void __launch_bounds__(WARPS * 32, RG * WARPS <= 8 ? 2 : 1)
latent_few_kernel(const __grid_constant__ CUtensorMap map, q38_latent_attention_params p, q38_batch_desc b, q38_kv_layer_desc kv,
                  int splits) {
  constexpr int ROWS = 16 * RG, KEYS_T = kPage * ROWS / (32 * WARPS);  // keys of a row that a thread of the softmax takes
  constexpr int ROW_T = kPage / KEYS_T;                                // threads of a row
  constexpr int KP = 16 / WARPS;                                       // 16-key pieces of a warp's scores
  static_assert(KEYS_T % 4 == 0 && ROW_T <= 32 && KP >= 1 && NT % 2 == 0, "shape");
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = ring_base(smem_raw);
  __shared__ __align__(8) uint64_t full[STAGES];
  __shared__ int issued[STAGES];
  __shared__ float factor[ROWS], row_m[ROWS], row_l[ROWS];
  const int k_dim = kv.k_dim;
  float* part = reinterpret_cast<float*>(smem + STAGES * page_smem(k_dim));  // [4 quarters][ROWS][kXS]
  bf16* p_hi = reinterpret_cast<bf16*>(part + 4 * ROWS * kXS);               // [ROWS][kPS]
  bf16* p_lo = p_hi + ROWS * kPS;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int split = blockIdx.y, seq = blockIdx.z;
  pdl_wait();
  pdl_launch_dependents();
  const int start = b.seq_start[seq], count = b.seq_start[seq + 1] - start, pos0 = b.seq_pos0[seq], H = p.heads;
  const Share sh = share_of(blockIdx.x, ROWS, count, H, pos0, split, splits);
  if (sh.p0 >= sh.p1) return;
  const PageRing<STAGES> ring{full, issued, smem, kv.block_table + (size_t)b.seq_slot[seq] * kv.max_pages_per_seq, k_dim, sh.p0, sh.p1};
  if (tid == 0) ring.start(&map, kv.num_pages);
  __syncthreads();

  // this warp's share of the queries: fragments of KS k16 steps, zero where there is no row or no dimension
  const int kg = warp & 3, key0 = (warp >> 2) * 16 * KP;
  const bf16* q = static_cast<const bf16*>(p.q) + ((size_t)start * H + sh.first) * k_dim;
  uint32_t qf[RG][KS][4];
#pragma unroll
  for (int r = 0; r < RG; ++r)
#pragma unroll
    for (int k = 0; k < KS; ++k)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int row = 16 * r + g + 8 * (e & 1), d = (kg * KS + k) * 16 + 2 * t4 + 8 * (e >> 1);
        qf[r][k][e] = row < sh.rows && d < k_dim ? *reinterpret_cast<const uint32_t*>(q + (size_t)row * k_dim + d) : 0u;
      }
  // this thread's row of the softmax
  const int srow = tid / ROW_T, skey = tid % ROW_T * 4;  // ... and of its keys: four from skey, four from skey + 4 ROW_T, ...
  const int spos = srow < sh.rows ? pos0 + (sh.first + srow) / H : -1;
  const float scale2 = p.scale * kLog2e;
  float m = -INFINITY, l = 0.0f;
  float o[RG][NT][4];
#pragma unroll
  for (int r = 0; r < RG; ++r)
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[r][i][e] = 0.0f;
  const int c0 = warp * NT * 8;
  uint32_t k_l[KS], v_l[NT / 2];  // this lane's rows of the fragments; sixteen latents further is 2048 bytes further
#pragma unroll
  for (int k = 0; k < KS; ++k) k_l[k] = page_at(key0 + (lane & 7) + ((lane >> 4) << 3), 2 * (kg * KS + k) + ((lane >> 3) & 1));
#pragma unroll
  for (int np = 0; np < NT / 2; ++np) v_l[np] = page_at((lane & 7) + (((lane >> 3) & 1) << 3), c0 / 8 + 2 * np + (lane >> 4));
  const uint32_t ph_a = smem_u32(p_hi) + uint32_t((lane & 15) * kPS + (lane >> 4) * 8) * 2, pl_a = ph_a + ROWS * kPS * 2;
  bool ok = true;

  for (int pg = sh.p0; pg < sh.p1; ++pg) {
    ok = ok && ring.wait(pg);
    const uint32_t c_a = ring.at(pg);
    // ---- this warp's part of the scores ----
    float s[RG][2 * KP][4] = {};
#pragma unroll
    for (int k = 0; k < KS; ++k) {
      if ((kg * KS + k) * 16 >= k_dim) break;
      uint32_t kf[KP][4];
#pragma unroll
      for (int x = 0; x < KP; ++x) ldmatrix_x4(kf[x], c_a + k_l[k] + uint32_t(x * 2048));
#pragma unroll
      for (int r = 0; r < RG; ++r)
#pragma unroll
        for (int x = 0; x < KP; ++x) {
          mma_bf16_16816(s[r][2 * x], qf[r][k], kf[x][0], kf[x][1]);
          mma_bf16_16816(s[r][2 * x + 1], qf[r][k], kf[x][2], kf[x][3]);
        }
    }
#pragma unroll
    for (int r = 0; r < RG; ++r)
#pragma unroll
      for (int kt = 0; kt < 2 * KP; ++kt)
#pragma unroll
        for (int hf = 0; hf < 2; ++hf)
          *reinterpret_cast<float2*>(part + (kg * ROWS + 16 * r + g + 8 * hf) * kXS + key0 + 8 * kt + 2 * t4) =
              make_float2(s[r][kt][2 * hf], s[r][kt][2 * hf + 1]);
    __syncthreads();
    // ---- softmax ----
    {
      float x[KEYS_T], top = -INFINITY;
#pragma unroll
      for (int i = 0; i < KEYS_T; i += 4) {
        float4 v = make_float4(0, 0, 0, 0);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const float4 y = *reinterpret_cast<const float4*>(part + (k * ROWS + srow) * kXS + skey + i * ROW_T);
          v.x += y.x;
          v.y += y.y;
          v.z += y.z;
          v.w += y.w;
        }
        x[i] = v.x;
        x[i + 1] = v.y;
        x[i + 2] = v.z;
        x[i + 3] = v.w;
      }
#pragma unroll
      for (int i = 0; i < KEYS_T; ++i) {
        x[i] = pg * kPage + skey + i / 4 * 4 * ROW_T + i % 4 <= spos ? x[i] * scale2 : -INFINITY;
        top = fmaxf(top, x[i]);
      }
#pragma unroll
      for (int d = 1; d < ROW_T; d <<= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, d));
      top = fmaxf(top, m);
      const float base = top == -INFINITY ? 0.0f : top, f = ex2(m - base);
      m = top;
      l *= f;
      if (skey == 0) factor[srow] = f;
#pragma unroll
      for (int i = 0; i < KEYS_T; i += 4) {
        __nv_bfloat162 hi[2], lo[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float w0 = ex2(x[i + 2 * e] - base), w1 = ex2(x[i + 2 * e + 1] - base);
          l += w0 + w1;
          hi[e] = __floats2bfloat162_rn(w0, w1);
          const float2 h = __bfloat1622float2(hi[e]);
          lo[e] = __floats2bfloat162_rn(w0 - h.x, w1 - h.y);
        }
        *reinterpret_cast<uint2*>(p_hi + srow * kPS + skey + i * ROW_T) = *reinterpret_cast<const uint2*>(hi);
        *reinterpret_cast<uint2*>(p_lo + srow * kPS + skey + i * ROW_T) = *reinterpret_cast<const uint2*>(lo);
      }
    }
    __syncthreads();
    // ---- outputs: all rows and keys, this warp's columns ----
#pragma unroll
    for (int r = 0; r < RG; ++r) {
      const float fa = factor[16 * r + g], fb = factor[16 * r + g + 8];
      if (__any_sync(0xffffffffu, fa != 1.0f || fb != 1.0f)) {
#pragma unroll
        for (int i = 0; i < NT; ++i) {
          o[r][i][0] *= fa;
          o[r][i][1] *= fa;
          o[r][i][2] *= fb;
          o[r][i][3] *= fb;
        }
      }
    }
    if (c0 < k_dim) {
#pragma unroll
      for (int kb = 0; kb < kPage / 16; ++kb) {
        uint32_t ph[RG][4], pl[RG][4], v[NT / 2][4];
#pragma unroll
        for (int r = 0; r < RG; ++r) {
          ldmatrix_x4(ph[r], ph_a + uint32_t(16 * r * kPS + kb * 16) * 2);
          ldmatrix_x4(pl[r], pl_a + uint32_t(16 * r * kPS + kb * 16) * 2);
        }
#pragma unroll
        for (int np = 0; np < NT / 2; ++np)
          if (c0 + 16 * np < k_dim) ldmatrix_x4_trans(v[np], c_a + v_l[np] + uint32_t(kb * 2048));
#pragma unroll
        for (int term = 0; term < 2; ++term)
#pragma unroll
          for (int r = 0; r < RG; ++r)
#pragma unroll
            for (int np = 0; np < NT / 2; ++np)
              if (c0 + 16 * np < k_dim) {
                mma_bf16_16816(o[r][2 * np], term ? ph[r] : pl[r], v[np][0], v[np][1]);
                mma_bf16_16816(o[r][2 * np + 1], term ? ph[r] : pl[r], v[np][2], v[np][3]);
              }
      }
    }
    if (pg + 1 < sh.p1) {
      __syncthreads();  // everybody is done with the page, the weights and the factors
      if (tid == 0 && ok && pg + STAGES < sh.p1) ring.load(&map, kv.num_pages, pg + STAGES);
    }
  }
#pragma unroll
  for (int d = 1; d < ROW_T; d <<= 1) l += __shfl_xor_sync(0xffffffffu, l, d);
  if (skey == 0) {
    row_m[srow] = m;
    row_l[srow] = l;
  }
  ring.finish(ok);
#pragma unroll
  for (int r = 0; r < RG; ++r)
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int row = 16 * r + g + 8 * hf;
      if (row >= sh.rows) continue;
      RowOut to{static_cast<bf16*>(p.out) + ((size_t)start * H + sh.first + row) * k_dim, nullptr, 1.0f / row_l[row]};
      if (splits > 1) to.rec = piece(p, k_dim, (size_t)seq * gridDim.x + blockIdx.x, split, splits, ROWS, row);
#pragma unroll
      for (int i = 0; i < NT; ++i)
        if (c0 + 8 * i < k_dim) to.put(c0 + 8 * i + 2 * t4, o[r][i][2 * hf], o[r][i][2 * hf + 1]);
      if (splits > 1 && warp == 0 && t4 == 0) *reinterpret_cast<float2*>(to.rec + k_dim) = make_float2(row_m[row], row_l[row]);
    }
}

// 64 rows, sixteen warps: four row groups x four column groups; a warp scores 16 keys of a page for its rows (queries from
// shared memory) and carries NT * 8 columns of their outputs.
constexpr int kManyThreads = 512, kManyRows = 64, kCG = 4;
template <int NT, int STAGES>
__global__ void __launch_bounds__(kManyThreads, 1)
latent_many_kernel(const __grid_constant__ CUtensorMap map, q38_latent_attention_params p, q38_batch_desc b, q38_kv_layer_desc kv,
                   int splits) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = ring_base(smem_raw);
  __shared__ __align__(8) uint64_t full[STAGES];
  __shared__ int issued[STAGES];
  __shared__ float mx[kManyRows][kCG], sum[kManyRows][kCG];
  const int k_dim = kv.k_dim, rs = row_stride(k_dim);
  bf16* q_s = reinterpret_cast<bf16*>(smem + STAGES * page_smem(k_dim));  // [64][rs]
  bf16* p_hi = q_s + kManyRows * rs;                                      // [64][kPS]
  bf16* p_lo = p_hi + kManyRows * kPS;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int rg = warp / kCG, cg = warp % kCG, split = blockIdx.y, seq = blockIdx.z;
  pdl_wait();
  pdl_launch_dependents();
  const int start = b.seq_start[seq], count = b.seq_start[seq + 1] - start, pos0 = b.seq_pos0[seq], H = p.heads;
  const Share sh = share_of(blockIdx.x, kManyRows, count, H, pos0, split, splits);
  if (sh.p0 >= sh.p1) return;
  const PageRing<STAGES> ring{full, issued, smem, kv.block_table + (size_t)b.seq_slot[seq] * kv.max_pages_per_seq, k_dim, sh.p0, sh.p1};
  if (tid == 0) ring.start(&map, kv.num_pages);
  __syncthreads();
  const uint4* q = reinterpret_cast<const uint4*>(static_cast<const bf16*>(p.q) + ((size_t)start * H + sh.first) * k_dim);
  const int pieces = k_dim / 8;
  for (int i = tid; i < kManyRows * pieces; i += kManyThreads)
    *reinterpret_cast<uint4*>(q_s + i / pieces * rs + i % pieces * 8) = i < sh.rows * pieces ? q[i] : make_uint4(0, 0, 0, 0);
  __syncthreads();

  const int ra = 16 * rg + g, rb = ra + 8;
  const int pos_a = ra < sh.rows ? pos0 + (sh.first + ra) / H : -1, pos_b = rb < sh.rows ? pos0 + (sh.first + rb) / H : -1;
  const float scale2 = p.scale * kLog2e;
  float m_a = -INFINITY, m_b = -INFINITY, l_a = 0.0f, l_b = 0.0f;
  float o[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[i][e] = 0.0f;
  const uint32_t q_a = smem_u32(q_s) + ((16 * rg + (lane & 15)) * rs + (lane >> 4) * 8) * 2;
  const uint32_t ph_a = smem_u32(p_hi) + ((16 * rg + (lane & 15)) * kPS + (lane >> 4) * 8) * 2, pl_a = ph_a + kManyRows * kPS * 2;
  const int c0 = cg * NT * 8, key0 = cg * 16;  // first output column and key of this warp
  bool ok = true;

  for (int pg = sh.p0; pg < sh.p1; ++pg) {
    ok = ok && ring.wait(pg);
    const uint32_t c_a = ring.at(pg);
    // ---- scores of this warp's keys, every other step into accumulators of its own ----
    float s[2][4] = {}, s2[2][4] = {};
    const int krow = key0 + (lane & 7) + ((lane >> 4) << 3), kchunk = (lane >> 3) & 1;
#pragma unroll 2
    for (int k = 0; k < k_dim; k += 32) {
      uint32_t a[2][4], kf[2][4];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        ldmatrix_x4(a[e], q_a + (k + 16 * e) * 2);
        ldmatrix_x4(kf[e], c_a + page_at(krow, k / 8 + 2 * e + kchunk));
      }
      mma_bf16_16816(s[0], a[0], kf[0][0], kf[0][1]);
      mma_bf16_16816(s[1], a[0], kf[0][2], kf[0][3]);
      mma_bf16_16816(s2[0], a[1], kf[1][0], kf[1][1]);
      mma_bf16_16816(s2[1], a[1], kf[1][2], kf[1][3]);
    }
    float ma = -INFINITY, mb = -INFINITY;
#pragma unroll
    for (int kt = 0; kt < 2; ++kt)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int key = pg * kPage + key0 + 8 * kt + 2 * t4 + e;
        s[kt][e] = key <= pos_a ? (s[kt][e] + s2[kt][e]) * scale2 : -INFINITY;
        s[kt][2 + e] = key <= pos_b ? (s[kt][2 + e] + s2[kt][2 + e]) * scale2 : -INFINITY;
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
    for (int x = 0; x < kCG; ++x) {
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
    for (int kt = 0; kt < 2; ++kt)
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const float base = hf ? base_b : base_a;
        const float w0 = ex2(s[kt][2 * hf] - base), w1 = ex2(s[kt][2 * hf + 1] - base);
        (hf ? l_b : l_a) += w0 + w1;
        const __nv_bfloat162 hi = __floats2bfloat162_rn(w0, w1);
        const float2 f = __bfloat1622float2(hi);
        const int at = (hf ? rb : ra) * kPS + key0 + 8 * kt + 2 * t4;
        *reinterpret_cast<__nv_bfloat162*>(p_hi + at) = hi;
        *reinterpret_cast<__nv_bfloat162*>(p_lo + at) = __floats2bfloat162_rn(w0 - f.x, w1 - f.y);
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
    uint32_t v_l[NT / 2];
#pragma unroll
    for (int np = 0; np < NT / 2; ++np) v_l[np] = c_a + page_at((lane & 7) + (((lane >> 3) & 1) << 3), c0 / 8 + 2 * np + (lane >> 4));
#pragma unroll
    for (int kb = 0; kb < kPage / 16; ++kb) {
      uint32_t ph[4], pl[4];
      ldmatrix_x4(ph, ph_a + kb * 32);
      ldmatrix_x4(pl, pl_a + kb * 32);
#pragma unroll
      for (int np = 0; np < NT / 2; np += 2) {  // four products between two that depend on one another
        if (c0 + 16 * np >= k_dim) break;
        uint32_t v[2][4];
#pragma unroll
        for (int x = 0; x < 2; ++x) ldmatrix_x4_trans(v[x], v_l[np + x] + uint32_t(kb * 2048));
#pragma unroll
        for (int term = 0; term < 2; ++term)
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            mma_bf16_16816(o[2 * (np + x)], term ? ph : pl, v[x][0], v[x][1]);
            mma_bf16_16816(o[2 * (np + x) + 1], term ? ph : pl, v[x][2], v[x][3]);
          }
      }
    }
    if (pg + 1 < sh.p1) {
      __syncthreads();  // everybody is done with the page, the weights and the maxima
      if (tid == 0 && ok && pg + STAGES < sh.p1) ring.load(&map, kv.num_pages, pg + STAGES);
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
  ring.finish(ok);
  l_a = l_b = 0.0f;
#pragma unroll
  for (int x = 0; x < kCG; ++x) {
    l_a += sum[ra][x];
    l_b += sum[rb][x];
  }
#pragma unroll
  for (int hf = 0; hf < 2; ++hf) {
    const int r = hf ? rb : ra;
    if (r >= sh.rows) continue;
    RowOut to{static_cast<bf16*>(p.out) + ((size_t)start * H + sh.first + r) * k_dim, nullptr, 1.0f / (hf ? l_b : l_a)};
    if (splits > 1) to.rec = piece(p, k_dim, (size_t)seq * gridDim.x + blockIdx.x, split, splits, kManyRows, r);
#pragma unroll
    for (int i = 0; i < NT; ++i)
      if (c0 + 8 * i < k_dim) to.put(c0 + 8 * i + 2 * t4, o[i][2 * hf], o[i][2 * hf + 1]);
    if (splits > 1 && cg == 0 && t4 == 0) *reinterpret_cast<float2*>(to.rec + k_dim) = make_float2(hf ? m_b : m_a, hf ? l_b : l_a);
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
#pragma unroll 8
    for (int s = 0; s < sh.active; ++s) {
      const float2 x = *reinterpret_cast<const float2*>(piece(p, k_dim, at, s, splits, block_rows, r) + c);
      v.x += factor[s] * x.x;
      v.y += factor[s] * x.y;
    }
    *reinterpret_cast<__nv_bfloat162*>(out + c) = __floats2bfloat162_rn(v.x, v.y);
  }
}

constexpr int kMaxKDim = 512, kMaxSplits = 64;
constexpr int kPieceRows = 64;  // rows of pieces per SM that the scratch holds

using MmaKernel = void (*)(CUtensorMap, q38_latent_attention_params, q38_batch_desc, q38_kv_layer_desc, int);
// `resident`: CTAs of the kernel that share an SM
int launch_mma(MmaKernel kernel, int threads, int block_rows, size_t smem, int resident, const q38_latent_attention_params& p,
               const q38_batch_desc& b, const q38_kv_layer_desc& kv, cudaStream_t s) {
  const int blocks = (b.max_tokens_per_seq * p.heads + block_rows - 1) / block_rows;
  const long long ctas = (long long)blocks * b.num_seqs;
  // Few CTAs: the pages of each over as many as there is room for (and scratch for the pieces).
  int splits = int(std::min<long long>(kMaxSplits, (long long)num_sms() * resident / ctas));
  const size_t per_split = size_t(ctas) * block_rows * size_t(kv.k_dim + 2);
  if (!p.partials) splits = 1;
  else splits = std::max(1, std::min(splits, int(std::min<size_t>(kMaxSplits, p.partial_floats / per_split))));
  CUtensorMap map;  // the layer's pages as one matrix of latents
  if (const int rc = encode_bf16_rows(&map, kv.pages, (long long)kv.num_pages * kPage, kv.k_dim, kv.k_dim, kPage)) return rc;
  (void)launch_kernel(kernel, dim3(blocks, splits, b.num_seqs), dim3(threads), smem, s, map, p, b, kv, splits);
  Q38_LAUNCH_OK("latent attention kernel");
  if (splits > 1) {
    (void)launch_kernel(latent_join_kernel, dim3(b.max_tokens_per_seq * p.heads, b.num_seqs), dim3(128), 0, s, p, b, kv.k_dim, blocks,
                        block_rows, splits);
    Q38_LAUNCH_OK("latent_join_kernel");
  }
  return Q38_OK;
}

constexpr int kStaticSmem = 3072;  // room left for the kernels' static shared memory
template <int RG, int WARPS, int KS, int STAGES>
int launch_few(const q38_latent_attention_params& p, const q38_batch_desc& b, const q38_kv_layer_desc& kv, cudaStream_t s) {
  constexpr int NT = KS * 8 / WARPS;  // four quarters of KS * 16 dimensions over all warps
  static const cudaError_t attr = cudaFuncSetAttribute(latent_few_kernel<RG, WARPS, KS, NT, STAGES>,
                                                       cudaFuncAttributeMaxDynamicSharedMemorySize, max_optin_smem() - kStaticSmem);
  Q38_CUDA_OK(attr);
  const size_t smem = 1024 + size_t(STAGES) * page_smem(kv.k_dim) + size_t(16 * RG) * (4 * kXS * 4 + 2 * kPS * 2);
  const int resident = smem < size_t(100) * 1024 && RG * WARPS <= 8 ? 2 : 1;
  return launch_mma(latent_few_kernel<RG, WARPS, KS, NT, STAGES>, 32 * WARPS, 16 * RG, smem, resident, p, b, kv, s);
}
template <int RG>
int launch_few_rows(const q38_latent_attention_params& p, const q38_batch_desc& b, const q38_kv_layer_desc& kv, cudaStream_t s) {
  // 16 rows: two CTAs per SM, which cover one another's loads where only one buffer fits
  if (kv.k_dim <= 128) return launch_few<RG, 8, 2, 3>(p, b, kv, s);
  if (kv.k_dim <= 256) return launch_few<RG, 8, 4, 2>(p, b, kv, s);
  return launch_few<RG, 8, 8, RG == 1 ? 1 : 2>(p, b, kv, s);
}
template <int NT>
int launch_many(const q38_latent_attention_params& p, const q38_batch_desc& b, const q38_kv_layer_desc& kv, cudaStream_t s) {
  static const cudaError_t attr =
      cudaFuncSetAttribute(latent_many_kernel<NT, 2>, cudaFuncAttributeMaxDynamicSharedMemorySize, max_optin_smem() - kStaticSmem);
  Q38_CUDA_OK(attr);
  const size_t smem = 1024 + size_t(2) * page_smem(kv.k_dim) + size_t(kManyRows) * (row_stride(kv.k_dim) + 2 * kPS) * 2;
  return launch_mma(latent_many_kernel<NT, 2>, kManyThreads, kManyRows, smem, 1, p, b, kv, s);
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
      kv->page_bytes != size_t(kPage) * kv->k_dim * 2)
    return launch_general<bf16>(*p, *batch, *kv, s);
  const int rows = batch->max_tokens_per_seq * p->heads;
  if (rows <= 16) return launch_few_rows<1>(*p, *batch, *kv, s);
  if (rows <= 32) return launch_few_rows<2>(*p, *batch, *kv, s);
  return kv->k_dim <= 128 ? launch_many<4>(*p, *batch, *kv, s)
         : kv->k_dim <= 256 ? launch_many<8>(*p, *batch, *kv, s) : launch_many<16>(*p, *batch, *kv, s);
}
