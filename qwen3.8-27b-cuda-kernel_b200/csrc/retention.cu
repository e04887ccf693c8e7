// Retention of the layer-list architectures: linear attention with a fixed decay per head,
//   S_t = decay S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,   out = silu(g) o / rms(o)  per head.
// q and k are rotated in fp32 from the projections' values and stay fp32; so do the state and o.
//
// Decode batches: one CTA per (head, sequence) streams the head's state through registers once, with rotation, norm and
//   output gate in the same kernel.
// Prefill (bf16 activations): three kernels. rope: rotated q and k as bf16 hi + lo terms (16 mantissa bits). chunk: a CTA
//   per (32 value columns, head, sequence) walks the run in chunks of 64 tokens with the state as fp32 MMA accumulators:
//     o_i = decay^(i+1) S^T q_i + sum_(j <= i) decay^(i-j) (q_i . k_j) v_j,   S' = decay^n S + sum_j decay^(n-1-j) k_j v_j^T,
//   every product on mma.sync with each fp32 factor as hi + lo (three MMAs per product, two where one factor is bf16).
//   gate: norm and output gate of each (token, head).
// Any size, fp32 activations: a kernel that walks the run token by token with 32 value columns of the state in shared memory.
#include <algorithm>

#include "act.cuh"
#include "host_util.h"

namespace q38 {
Q38_REGISTER_ERROR_WORD();
namespace {

using bf16 = __nv_bfloat16;
constexpr int kChunk = Q38_RETENTION_CHUNK;
__host__ __device__ constexpr int up16(int x) { return (x + 15) / 16 * 16; }

// cos and sin of position * inv_freq; the angle is formed and reduced in double precision
__device__ __forceinline__ float2 turn_of(int pos, double inv_freq) {
  const double turns = double(pos) * inv_freq * 0.15915494309189535;
  float sn, cs;
  sincosf(float((turns - rint(turns)) * 6.283185307179586), &sn, &cs);
  return make_float2(cs, sn);
}
// element d of a rotated head
template <typename T>
__device__ __forceinline__ float rotated(const T* h, int d, int half, const float2* trig) {
  const float y = to_f32(h[d]);
  if (d >= 2 * half) return y;
  const float2 t = trig[d < half ? d : d - half];
  return d < half ? y * t.x - to_f32(h[d + half]) * t.y : y * t.x + to_f32(h[d - half]) * t.y;
}

// ---- token by token, any size -------------------------------------------------------------------------------------------
constexpr int kSeqCols = 32, kSeqWarps = 8;
template <typename T>
__global__ void __launch_bounds__(kSeqCols * kSeqWarps)
retention_sequential_kernel(q38_retention_params p, q38_batch_desc b, q38_recurrent_state_desc st) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ __align__(16) float sm[];
  const int half = p.rot_dims / 2;
  float2* trig = reinterpret_cast<float2*>(sm);     // [half]
  float* S = sm + 2 * half;                         // [dim][32]
  float* q_sm = S + p.dim * kSeqCols;               // [dim]
  float* k_sm = q_sm + p.dim;
  __shared__ float red[kSeqWarps][kSeqCols];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, h = blockIdx.y, seq = blockIdx.z;
  const int c = blockIdx.x * kSeqCols + lane;
  const bool live = c < p.vdim;
  const int start = b.seq_start[seq], count = b.seq_start[seq + 1] - start, pos0 = b.seq_pos0[seq];
  float* state = reinterpret_cast<float*>(st.state + (size_t)b.seq_slot[seq] * st.slot_bytes) + (size_t)h * p.dim * p.vdim;
  const float decay = p.decay_pow[h * (kChunk + 1) + 1];
  for (int d = warp; d < p.dim; d += kSeqWarps) S[d * kSeqCols + lane] = live && pos0 > 0 ? state[(size_t)d * p.vdim + c] : 0.0f;
  for (int t = 0; t < count; ++t) {
    const T* row = static_cast<const T*>(p.proj) + (size_t)(start + t) * p.ld_proj;
    for (int i = threadIdx.x; i < half; i += blockDim.x) trig[i] = turn_of(pos0 + t, p.inv_freq[i]);
    __syncthreads();
    for (int d = threadIdx.x; d < p.dim; d += blockDim.x) {
      q_sm[d] = rotated(row + (size_t)h * p.dim, d, half, trig);
      k_sm[d] = rotated(row + (size_t)(p.heads + h) * p.dim, d, half, trig) * p.k_scale;
    }
    const float v = live ? to_f32(row[(size_t)2 * p.heads * p.dim + (size_t)h * p.vdim + c]) : 0.0f;
    __syncthreads();
    float o = 0.0f;
    for (int d = warp; d < p.dim; d += kSeqWarps) {
      const float s = decay * S[d * kSeqCols + lane] + k_sm[d] * v;
      S[d * kSeqCols + lane] = s;
      o += q_sm[d] * s;
    }
    red[warp][lane] = o;
    __syncthreads();
    if (warp == 0 && live) {
      float total = 0.0f;
#pragma unroll
      for (int w = 0; w < kSeqWarps; ++w) total += red[w][lane];
      p.o[(size_t)(start + t) * p.heads * p.vdim + (size_t)h * p.vdim + c] = total;
    }
  }
  if (live && count > 0)
    for (int d = warp; d < p.dim; d += kSeqWarps) state[(size_t)d * p.vdim + c] = S[d * kSeqCols + lane];
}

// norm and output gate: one warp per (token, head)
template <typename T>
__global__ void __launch_bounds__(256) retention_gate_kernel(q38_retention_params p, q38_batch_desc b) {
  pdl_wait();
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31, item = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (item >= b.num_tokens * p.heads) return;
  const int row = b.seq_start[0] + item / p.heads, h = item % p.heads;
  const float* o = p.o + ((size_t)row * p.heads + h) * p.vdim;
  const T* g = static_cast<const T*>(p.proj) + (size_t)row * p.ld_proj + (size_t)p.heads * (2 * p.dim + p.vdim) + (size_t)h * p.vdim;
  T* out = static_cast<T*>(p.out) + (size_t)row * p.ld_out + (size_t)h * p.vdim;
  float ss = 0.0f;
  for (int c = lane; c < p.vdim; c += 32) ss += o[c] * o[c];
  const float rs = 1.0f / sqrtf(warp_sum(ss) / float(p.vdim) + p.eps);
  for (int c = lane; c < p.vdim; c += 32) out[c] = from_f32<T>(o[c] * rs * silu_f(to_f32(g[c])));
}

// ---- decode batches ----------------------------------------------------------------------------------------------------------
constexpr int kDecThreads = 256, kDecBatch = 8;
template <typename T>
__global__ void __launch_bounds__(kDecThreads)
retention_decode_kernel(q38_retention_params p, q38_batch_desc b, q38_recurrent_state_desc st) {
  extern __shared__ __align__(16) float sm[];
  const int half = p.rot_dims / 2, v4 = p.vdim / 4, rows = kDecThreads / v4;  // state rows in flight per round
  float* red = sm;                                           // [rows][vdim]
  float2* trig = reinterpret_cast<float2*>(red + rows * p.vdim);
  float* q_sm = reinterpret_cast<float*>(trig + half);
  float* k_sm = q_sm + p.dim;
  __shared__ float red_ss[33];
  const int h = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x, r = tid / v4, c = tid % v4;
  const bool live = r < rows;
  pdl_wait();
  pdl_launch_dependents();
  float4* state = reinterpret_cast<float4*>(st.state + (size_t)b.seq_slot[seq] * st.slot_bytes) + (size_t)h * p.dim * v4 + c;
  const int rounds = (p.dim + rows - 1) / rows;
  const int start = b.seq_start[seq], pos = b.seq_pos0[seq];
  const bool fresh = pos == 0;
  float4 s[kDecBatch];
  auto load = [&](int i0) {
#pragma unroll
    for (int i = 0; i < kDecBatch; ++i) {
      const int d = (i0 + i) * rows + r;
      s[i] = live && !fresh && d < p.dim ? state[(size_t)d * v4] : make_float4(0, 0, 0, 0);
    }
  };
  load(0);  // in flight while the query and the key are rotated
  const float decay = p.decay_pow[h * (kChunk + 1) + 1];
  const T* row = static_cast<const T*>(p.proj) + (size_t)start * p.ld_proj;
  for (int i = tid; i < half; i += kDecThreads) trig[i] = turn_of(pos, p.inv_freq[i]);
  float4 v = make_float4(0, 0, 0, 0), o = v;
  if (live) {
    const T* vr = row + (size_t)2 * p.heads * p.dim + (size_t)h * p.vdim + 4 * c;
    v = make_float4(to_f32(vr[0]), to_f32(vr[1]), to_f32(vr[2]), to_f32(vr[3]));
  }
  __syncthreads();
  for (int d = tid; d < p.dim; d += kDecThreads) {
    q_sm[d] = rotated(row + (size_t)h * p.dim, d, half, trig);
    k_sm[d] = rotated(row + (size_t)(p.heads + h) * p.dim, d, half, trig) * p.k_scale;
  }
  __syncthreads();
  for (int i0 = 0; i0 < rounds; i0 += kDecBatch) {
    if (i0 > 0) load(i0);
#pragma unroll
    for (int i = 0; i < kDecBatch; ++i) {
      const int d = (i0 + i) * rows + r;
      if (!live || d >= p.dim) continue;
      const float k = k_sm[d], q = q_sm[d];
      s[i].x = decay * s[i].x + k * v.x;
      s[i].y = decay * s[i].y + k * v.y;
      s[i].z = decay * s[i].z + k * v.z;
      s[i].w = decay * s[i].w + k * v.w;
      state[(size_t)d * v4] = s[i];
      o.x += q * s[i].x;
      o.y += q * s[i].y;
      o.z += q * s[i].z;
      o.w += q * s[i].w;
    }
  }
  if (live) *reinterpret_cast<float4*>(red + r * p.vdim + 4 * c) = o;
  __syncthreads();
  // one column per thread and turn from here on
  const T* g = row + (size_t)p.heads * (2 * p.dim + p.vdim) + (size_t)h * p.vdim;
  float ss = 0.0f;
  for (int i = tid; i < p.vdim; i += kDecThreads) {
    float t = 0.0f;
    for (int k = 0; k < rows; ++k) t += red[k * p.vdim + i];
    red[i] = t;
    ss += t * t;
  }
  const float rs = 1.0f / sqrtf(block_sum(ss, red_ss) / float(p.vdim) + p.eps);
  T* out = static_cast<T*>(p.out) + (size_t)start * p.ld_out + (size_t)h * p.vdim;
  for (int i = tid; i < p.vdim; i += kDecThreads) out[i] = from_f32<T>(red[i] * rs * silu_f(to_f32(g[i])));
}

// ---- prefill on the tensor cores ---------------------------------------------------------------------------------------------
// scratch row of one (token, head): [q hi | q lo | k hi | k lo], each dim rounded up to 16, zero beyond dim
__global__ void __launch_bounds__(256) retention_rope_kernel(q38_retention_params p, q38_batch_desc b) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ __align__(16) float sm[];
  float2* trig = reinterpret_cast<float2*>(sm);
  const int half = p.rot_dims / 2, dp = up16(p.dim), row = b.seq_start[0] + blockIdx.x, pos = b.tok_pos[blockIdx.x];
  for (int i = threadIdx.x; i < half; i += blockDim.x) trig[i] = turn_of(pos, p.inv_freq[i]);
  __syncthreads();
  const bf16* in = static_cast<const bf16*>(p.proj) + (size_t)row * p.ld_proj;
  bf16* qk = static_cast<bf16*>(p.qk) + (size_t)row * p.heads * 4 * dp;
  const int pairs = dp / 2;
  for (int i = threadIdx.x; i < 2 * p.heads * pairs; i += blockDim.x) {
    const int hh = i / pairs, d = 2 * (i % pairs);  // hh: query heads, then key heads
    const bool key = hh >= p.heads;
    float y[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      y[e] = d + e < p.dim ? rotated(in + (size_t)hh * p.dim, d + e, half, trig) : 0.0f;
      if (key) y[e] *= p.k_scale;
    }
    const __nv_bfloat162 hi = __floats2bfloat162_rn(y[0], y[1]);
    const float2 f = __bfloat1622float2(hi);
    bf16* dst = qk + (size_t)(key ? hh - p.heads : hh) * 4 * dp + (key ? 2 * dp : 0) + d;
    *reinterpret_cast<__nv_bfloat162*>(dst) = hi;
    *reinterpret_cast<__nv_bfloat162*>(dst + dp) = __floats2bfloat162_rn(y[0] - f.x, y[1] - f.y);
  }
}

__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool real) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(real ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ uint32_t pack2(float a, float b) {
  const __nv_bfloat162 p = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&p);
}
// x as hi + lo, two neighbours at a time
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 f = __bfloat1622float2(h);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = pack2(a - f.x, b - f.y);
}

// one 16 x 16 block against 32 columns; consecutive products are independent of one another
__device__ __forceinline__ void mma_row(float (&d)[4][4], const uint32_t (&a)[4], const uint32_t (&b)[2][4]) {
#pragma unroll
  for (int np = 0; np < 2; ++np)
#pragma unroll
    for (int e = 0; e < 2; ++e) mma_bf16_16816(d[2 * np + e], a, b[np][2 * e], b[np][2 * e + 1]);
}

constexpr int kMmaThreads = 256, kVT = 32;  // value columns per CTA
constexpr int kVS = kVT + 8;                // row strides whose ldmatrix phases do not collide: odd multiples of 16 bytes
constexpr int kXS = kVT / 2 + 4;
struct ChunkSmem {
  int qk_stride, qk, v, s_hi, s_lo, w_hi, w_lo, x, pw, total;  // byte offsets
  __host__ __device__ ChunkSmem(int dp, int stages) {
    qk_stride = 4 * dp + 8;
    int at = 0;
    auto take = [&](int bytes) {
      const int here = at;
      at += (bytes + 15) / 16 * 16;
      return here;
    };
    qk = take(stages * kChunk * qk_stride * 2);
    v = take(stages * kChunk * kVS * 2);
    s_hi = take(dp * kVS * 2);
    s_lo = take(dp * kVS * 2);
    w_hi = take(kChunk * kVS * 2);
    w_lo = take(kChunk * kVS * 2);
    x = take(2 * kChunk * kXS * 4);
    pw = take((kChunk + 1) * 4);
    total = at;
  }
};

// ITEMS: 16-row blocks of the state per warp (dim up to 128 * ITEMS)
template <int ITEMS, int STAGES>
__global__ void __launch_bounds__(kMmaThreads, 1)
retention_chunk_kernel(q38_retention_params p, q38_batch_desc b, q38_recurrent_state_desc st, int vec) {
  extern __shared__ __align__(16) uint8_t smem[];
  const int dp = up16(p.dim);
  const ChunkSmem L(dp, STAGES);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int v0 = blockIdx.x * kVT, h = blockIdx.y, seq = blockIdx.z;
  float* pw = reinterpret_cast<float*>(smem + L.pw);
  for (int i = tid; i <= kChunk; i += kMmaThreads) pw[i] = p.decay_pow[h * (kChunk + 1) + i];
  pdl_wait();
  pdl_launch_dependents();
  const int start = b.seq_start[seq], count = b.seq_start[seq + 1] - start, pos0 = b.seq_pos0[seq];
  if (count <= 0) return;
  float* state = reinterpret_cast<float*>(st.state + (size_t)b.seq_slot[seq] * st.slot_bytes) + (size_t)h * p.dim * p.vdim;
  const int dblocks = dp / 16;

  // state accumulators: item i = rows 16 (warp + 8 i) + {g, g + 8}, columns v0 + 8 nt + 2 t4 + {0, 1}
  float S[ITEMS][4][4];
#pragma unroll
  for (int i = 0; i < ITEMS; ++i)
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = 16 * (warp + 8 * i) + g + 8 * (e >> 1), c = v0 + 8 * nt + 2 * t4 + (e & 1);
        S[i][nt][e] = pos0 > 0 && d < p.dim && c < p.vdim ? state[(size_t)d * p.vdim + c] : 0.0f;
      }

  const int chunks = (count + kChunk - 1) / kChunk;
  const bf16* qk_g = static_cast<const bf16*>(p.qk) + ((size_t)start * p.heads + h) * 4 * dp;
  const size_t qk_row = (size_t)p.heads * 4 * dp;
  const bf16* v_g = static_cast<const bf16*>(p.proj) + (size_t)start * p.ld_proj + (size_t)2 * p.heads * p.dim + (size_t)h * p.vdim + v0;
  const int pieces = dp / 2;  // 16-byte pieces of a scratch row
  auto load = [&](int c) {
    const int first = c * kChunk, n = min(kChunk, count - first), stage = c % STAGES;
    bf16* qk_s = reinterpret_cast<bf16*>(smem + L.qk) + (size_t)stage * kChunk * L.qk_stride;
    for (int i = tid; i < kChunk * pieces; i += kMmaThreads) {
      const int r = i / pieces, k = i % pieces;
      cp_async16(qk_s + r * L.qk_stride + 8 * k, qk_g + (size_t)(first + min(r, n - 1)) * qk_row + 8 * k, r < n);
    }
    bf16* v_s = reinterpret_cast<bf16*>(smem + L.v) + (size_t)stage * kChunk * kVS;
    if (vec) {
      for (int i = tid; i < kChunk * (kVT / 8); i += kMmaThreads) {
        const int r = i / (kVT / 8), k = i % (kVT / 8);
        const bool real = r < n && v0 + 8 * k < p.vdim;
        cp_async16(v_s + r * kVS + 8 * k, real ? v_g + (size_t)(first + r) * p.ld_proj + 8 * k : v_g, real);
      }
    } else {
      for (int i = tid; i < kChunk * kVT; i += kMmaThreads) {
        const int r = i / kVT, k = i % kVT;
        v_s[r * kVS + k] = r < n && v0 + k < p.vdim ? v_g[(size_t)(first + r) * p.ld_proj + k] : __float2bfloat16_rn(0.0f);
      }
    }
    cp_async_commit();
  };
  load(0);

  const int rg = warp & 3, half = warp >> 2;  // output rows 16 rg ..; this warp's share of the keys and of the state rows
  const uint32_t a_lane = uint32_t(lane & 15), a_col = uint32_t(lane >> 4) * 8;                                // A, row-major
  const uint32_t n_row = uint32_t((lane & 7) + ((lane >> 4) << 3)), n_col = uint32_t((lane >> 3) & 1) * 8;     // B from [n][k]
  const uint32_t k_row = uint32_t((lane & 7) + (((lane >> 3) & 1) << 3)), k_col = uint32_t(lane >> 4) * 8;     // B from [k][n]
  const uint32_t t_row = uint32_t((lane & 7) + ((lane >> 4) << 3)), t_col = uint32_t((lane >> 3) & 1) * 8;     // A from [k][m]
  const uint32_t sh_a = smem_u32(smem + L.s_hi), sl_a = smem_u32(smem + L.s_lo);
  const uint32_t wh_a = smem_u32(smem + L.w_hi), wl_a = smem_u32(smem + L.w_lo);
  float* X = reinterpret_cast<float*>(smem + L.x);  // [2 column halves][64][kXS]: partial outputs handed to the other warp

  for (int c = 0; c < chunks; ++c) {
    const int first = c * kChunk, n = min(kChunk, count - first), stage = c % STAGES;
    cp_async_wait<0>();
    __syncthreads();  // the chunk's rows have landed; everybody is done with the previous chunk
    if (STAGES > 1 && c + 1 < chunks) load(c + 1);
    const bf16* v_s = reinterpret_cast<const bf16*>(smem + L.v) + (size_t)stage * kChunk * kVS;
    const uint32_t qk_a = smem_u32(smem + L.qk) + uint32_t(stage * kChunk * L.qk_stride) * 2, v_a = smem_u32(v_s);
    // the state as hi + lo, and the values weighted for the state update
#pragma unroll
    for (int i = 0; i < ITEMS; ++i) {
      const int db = warp + 8 * i;
      if (db >= dblocks) break;
#pragma unroll
      for (int nt = 0; nt < 4; ++nt)
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
          uint32_t hi, lo;
          split2(S[i][nt][2 * hf], S[i][nt][2 * hf + 1], hi, lo);
          const int at = ((16 * db + g + 8 * hf) * kVS + 8 * nt + 2 * t4) * 2;
          *reinterpret_cast<uint32_t*>(smem + L.s_hi + at) = hi;
          *reinterpret_cast<uint32_t*>(smem + L.s_lo + at) = lo;
        }
    }
    for (int i = tid; i < kChunk * (kVT / 2); i += kMmaThreads) {
      const int r = i / (kVT / 2), k = 2 * (i % (kVT / 2));
      const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(v_s + r * kVS + k));
      const float w = r < n ? pw[n - 1 - r] : 0.0f;
      uint32_t hi, lo;
      split2(v.x * w, v.y * w, hi, lo);
      *reinterpret_cast<uint32_t*>(smem + L.w_hi + (r * kVS + k) * 2) = hi;
      *reinterpret_cast<uint32_t*>(smem + L.w_lo + (r * kVS + k) * 2) = lo;
    }
    __syncthreads();

    // ---- outputs: this warp's rows against half of the state rows and half of the 16-key blocks, all 32 columns ----
    float o[4][4] = {};
    const bool rows_live = 16 * rg < n;
    if (rows_live) {
      const uint32_t q_hi = qk_a + ((16 * rg + a_lane) * L.qk_stride + a_col) * 2, q_lo = q_hi + dp * 2;
      for (int kb = half; kb < dblocks; kb += 2) {
        uint32_t qh[4], ql[4];
        ldmatrix_x4(qh, q_hi + kb * 32);
        ldmatrix_x4(ql, q_lo + kb * 32);
        uint32_t sh[2][4], sl[2][4];
#pragma unroll
        for (int np = 0; np < 2; ++np) {
          const uint32_t at = ((16 * kb + k_row) * kVS + 16 * np + k_col) * 2;
          ldmatrix_x4_trans(sh[np], sh_a + at);
          ldmatrix_x4_trans(sl[np], sl_a + at);
        }
        mma_row(o, ql, sh);
        mma_row(o, qh, sl);
        mma_row(o, qh, sh);
      }
      const float fa = pw[16 * rg + g + 1], fb = pw[16 * rg + g + 9];
#pragma unroll
      for (int nt = 0; nt < 4; ++nt) {
        o[nt][0] *= fa;
        o[nt][1] *= fa;
        o[nt][2] *= fb;
        o[nt][3] *= fb;
      }
      for (int jb = half; jb <= rg; jb += 2) {
        float s[2][4] = {}, s_lh[2][4] = {}, s_hl[2][4] = {};  // the terms apart: chains of their own
        const uint32_t k_hi = qk_a + ((16 * jb + n_row) * L.qk_stride + 2 * dp + n_col) * 2, k_lo = k_hi + dp * 2;
        for (int kb = 0; kb < dblocks; ++kb) {
          uint32_t qh[4], ql[4], kh[4], kl[4];
          ldmatrix_x4(qh, q_hi + kb * 32);
          ldmatrix_x4(ql, q_lo + kb * 32);
          ldmatrix_x4(kh, k_hi + kb * 32);
          ldmatrix_x4(kl, k_lo + kb * 32);
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            mma_bf16_16816(s_lh[e], ql, kh[2 * e], kh[2 * e + 1]);
            mma_bf16_16816(s_hl[e], qh, kl[2 * e], kl[2 * e + 1]);
            mma_bf16_16816(s[e], qh, kh[2 * e], kh[2 * e + 1]);
          }
        }
#pragma unroll
        for (int e = 0; e < 2; ++e)
#pragma unroll
          for (int x = 0; x < 4; ++x) s[e][x] += s_lh[e][x] + s_hl[e][x];
        uint32_t ah[4], al[4];
#pragma unroll
        for (int e = 0; e < 2; ++e)
#pragma unroll
          for (int hf = 0; hf < 2; ++hf) {
            const int i = 16 * rg + g + 8 * hf, j = 16 * jb + 8 * e + 2 * t4;
            const float a0 = j <= i ? s[e][2 * hf] * pw[i - j] : 0.0f;
            const float a1 = j + 1 <= i ? s[e][2 * hf + 1] * pw[i - j - 1] : 0.0f;
            split2(a0, a1, ah[2 * e + hf], al[2 * e + hf]);
          }
        uint32_t v[2][4];
#pragma unroll
        for (int np = 0; np < 2; ++np) ldmatrix_x4_trans(v[np], v_a + ((16 * jb + k_row) * kVS + 16 * np + k_col) * 2);
        mma_row(o, al, v);
        mma_row(o, ah, v);
      }
      // the two warps of a row block swap halves: warp `half` finishes columns 16 half .. 16 half + 15
      float* mine = X + (size_t)(1 - half) * kChunk * kXS;
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
          const float x0 = half == 0 ? o[nt + 2][2 * hf] : o[nt][2 * hf], x1 = half == 0 ? o[nt + 2][2 * hf + 1] : o[nt][2 * hf + 1];
          *reinterpret_cast<float2*>(mine + (16 * rg + g + 8 * hf) * kXS + 8 * nt + 2 * t4) = make_float2(x0, x1);
        }
    }

    // ---- state: decay^n S + K^T W ----
    const float gn = pw[n];
#pragma unroll
    for (int i = 0; i < ITEMS; ++i) {
      const int db = warp + 8 * i;
      if (db >= dblocks) break;
#pragma unroll
      for (int nt = 0; nt < 4; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[i][nt][e] *= gn;
      const int jbs = (n + 15) / 16;
      for (int jb = 0; jb < jbs; ++jb) {
        uint32_t kh[4], kl[4];
        const uint32_t at = qk_a + ((16 * jb + t_row) * L.qk_stride + 2 * dp + 16 * db + t_col) * 2;
        ldmatrix_x4_trans(kh, at);
        ldmatrix_x4_trans(kl, at + dp * 2);
        uint32_t wh[2][4], wl[2][4];
#pragma unroll
        for (int np = 0; np < 2; ++np) {
          const uint32_t wat = ((16 * jb + k_row) * kVS + 16 * np + k_col) * 2;
          ldmatrix_x4_trans(wh[np], wh_a + wat);
          ldmatrix_x4_trans(wl[np], wl_a + wat);
        }
        mma_row(S[i], kl, wh);
        mma_row(S[i], kh, wl);
        mma_row(S[i], kh, wh);
      }
    }
    __syncthreads();  // the partial outputs are in X
    if (rows_live) {
      const float* theirs = X + (size_t)half * kChunk * kXS;
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
          const int r = 16 * rg + g + 8 * hf, col = 8 * nt + 2 * t4;
          if (r >= n) continue;
          const float2 x = *reinterpret_cast<const float2*>(theirs + r * kXS + col);
          const float y0 = x.x + (half == 0 ? o[nt][2 * hf] : o[nt + 2][2 * hf]);
          const float y1 = x.y + (half == 0 ? o[nt][2 * hf + 1] : o[nt + 2][2 * hf + 1]);
          const int vc = v0 + 16 * half + col;
          float* out = p.o + ((size_t)(start + first + r) * p.heads + h) * p.vdim + vc;
          if (vc + 1 < p.vdim && (p.vdim & 1) == 0) *reinterpret_cast<float2*>(out) = make_float2(y0, y1);
          else {
            if (vc < p.vdim) out[0] = y0;
            if (vc + 1 < p.vdim) out[1] = y1;
          }
        }
    }
    if (STAGES == 1 && c + 1 < chunks) {  // the only buffer: nobody may still be reading it
      __syncthreads();
      load(c + 1);
    }
  }
#pragma unroll
  for (int i = 0; i < ITEMS; ++i)
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = 16 * (warp + 8 * i) + g + 8 * (e >> 1), cc = v0 + 8 * nt + 2 * t4 + (e & 1);
        if (d < p.dim && cc < p.vdim) state[(size_t)d * p.vdim + cc] = S[i][nt][e];
      }
}

// ---- launchers -------------------------------------------------------------------------------------------------------------------
template <int ITEMS, int STAGES>
int launch_chunk(const q38_retention_params& p, const q38_batch_desc& b, const q38_recurrent_state_desc& st, cudaStream_t s) {
  static const cudaError_t attr = cudaFuncSetAttribute(retention_chunk_kernel<ITEMS, STAGES>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                       max_optin_smem());
  Q38_CUDA_OK(attr);
  const ChunkSmem L(up16(p.dim), STAGES);
  const int vec = p.vdim % 8 == 0 && (2 * p.heads * p.dim) % 8 == 0 && p.ld_proj % 8 == 0 && reinterpret_cast<uintptr_t>(p.proj) % 16 == 0;
  (void)launch_kernel(retention_chunk_kernel<ITEMS, STAGES>, dim3((p.vdim + kVT - 1) / kVT, p.heads, b.num_seqs), dim3(kMmaThreads),
                      size_t(L.total), s, p, b, st, vec);
  Q38_LAUNCH_OK("retention_chunk_kernel");
  return Q38_OK;
}

bool chunk_fits(const q38_retention_params& p) {
  return p.act == Q38_ACT_BF16 && p.dim <= 256 && ChunkSmem(up16(p.dim), 1).total <= max_optin_smem() &&
         p.ld_proj % 2 == 0 && reinterpret_cast<uintptr_t>(p.qk) % 16 == 0;
}

int launch_prefill_mma(const q38_retention_params& p, const q38_batch_desc& b, const q38_recurrent_state_desc& st, cudaStream_t s) {
  (void)launch_kernel(retention_rope_kernel, dim3(b.num_tokens), dim3(256), size_t(std::max(2, p.rot_dims)) * 4, s, p, b);
  Q38_LAUNCH_OK("retention_rope_kernel");
  const bool two = ChunkSmem(up16(p.dim), 2).total <= max_optin_smem();
  if (p.dim <= 128) return two ? launch_chunk<1, 2>(p, b, st, s) : launch_chunk<1, 1>(p, b, st, s);
  return two ? launch_chunk<2, 2>(p, b, st, s) : launch_chunk<2, 1>(p, b, st, s);
}

size_t decode_smem(const q38_retention_params& p) {
  const int rows = kDecThreads / (p.vdim / 4);
  return (size_t(rows) * p.vdim + size_t(p.rot_dims) + 2 * size_t(p.dim)) * 4;
}

template <typename T>
int launch_retention(const q38_retention_params& p, const q38_batch_desc& b, const q38_recurrent_state_desc& st, cudaStream_t s) {
  if (b.max_tokens_per_seq == 1 && p.vdim % 4 == 0 && p.vdim <= 4 * kDecThreads && p.rot_dims % 2 == 0 && st.slot_bytes % 16 == 0 &&
      reinterpret_cast<uintptr_t>(st.state) % 16 == 0 && decode_smem(p) <= 48 * 1024) {
    (void)launch_kernel(retention_decode_kernel<T>, dim3(p.heads, b.num_seqs), dim3(kDecThreads), decode_smem(p), s, p, b, st);
    Q38_LAUNCH_OK("retention_decode_kernel");
    return Q38_OK;
  }
  Q38_REQUIRE(p.o, "retention: scratch needed");
  if (chunk_fits(p) && p.qk && b.max_tokens_per_seq > 1) {
    if (const int rc = launch_prefill_mma(p, b, st, s)) return rc;
  } else {
    const size_t smem = (size_t(p.rot_dims) + size_t(p.dim) * (kSeqCols + 2)) * 4;
    Q38_REQUIRE(smem <= size_t(max_optin_smem()), "retention: heads of %d dimensions do not fit", p.dim);
    static const cudaError_t attr =
        cudaFuncSetAttribute(retention_sequential_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, max_optin_smem() - 2048);
    Q38_CUDA_OK(attr);
    Q38_REQUIRE(smem <= size_t(max_optin_smem() - 2048), "retention: heads of %d dimensions do not fit", p.dim);
    (void)launch_kernel(retention_sequential_kernel<T>, dim3((p.vdim + kSeqCols - 1) / kSeqCols, p.heads, b.num_seqs),
                        dim3(kSeqCols * kSeqWarps), smem, s, p, b, st);
    Q38_LAUNCH_OK("retention_sequential_kernel");
  }
  (void)launch_kernel(retention_gate_kernel<T>, dim3((b.num_tokens * p.heads + 7) / 8), dim3(256), 0, s, p, b);
  Q38_LAUNCH_OK("retention_gate_kernel");
  return Q38_OK;
}

}  // namespace
}  // namespace q38

using namespace q38;

extern "C" size_t q38_retention_qk_bytes(int tokens, int heads, int dim, int act) {
  return act == Q38_ACT_BF16 ? size_t(tokens) * size_t(heads) * 4 * size_t(up16(dim)) * 2 : 0;
}

extern "C" int q38_retention(const q38_retention_params* p, const q38_batch_desc* batch, const q38_recurrent_state_desc* st,
                             void* stream) {
  Q38_REQUIRE(p && batch && st && p->proj && p->out && p->decay_pow && st->state, "retention: null argument");
  if (batch->num_tokens == 0) return Q38_OK;
  Q38_REQUIRE(batch->seq_start && batch->seq_slot && batch->seq_pos0 && batch->tok_pos && batch->num_seqs > 0 &&
                  batch->num_seqs <= 65535 && batch->max_tokens_per_seq > 0, "retention: batch");
  Q38_REQUIRE(p->heads > 0 && p->heads <= 65535 && p->dim > 0 && p->vdim > 0, "retention: %d heads of %d x %d", p->heads, p->dim, p->vdim);
  Q38_REQUIRE(p->rot_dims >= 0 && p->rot_dims % 2 == 0 && p->rot_dims <= p->dim && p->rot_dims <= 4096 && (p->rot_dims == 0 || p->inv_freq),
              "retention: rot_dims %d", p->rot_dims);
  Q38_REQUIRE(p->ld_proj >= 2 * p->heads * (p->dim + p->vdim) && p->ld_out >= p->heads * p->vdim, "retention: leading dimensions");
  Q38_REQUIRE(p->act == Q38_ACT_BF16 || p->act == Q38_ACT_F32, "retention: activation precision %d", p->act);
  return p->act == Q38_ACT_BF16 ? launch_retention<__nv_bfloat16>(*p, *batch, *st, as_stream(stream))
                                : launch_retention<float>(*p, *batch, *st, as_stream(stream));
}
