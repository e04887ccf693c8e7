// Dense bf16 GEMM on the 5th-generation tensor cores (tcgen05.mma, accumulators in TMEM), any number of tokens.
//
// Orientation as in the BQ kernel: the weights are the MMA's A operand (128 output columns fill the 128 TMEM lanes), the
// tokens its N operand (TOK = 32 ... 256). Both operands arrive by TMA (2-D tensor maps, 128-byte swizzle; rows and
// columns outside the matrices are zero-filled, so any n, k and m work) into a ring of stages of one 64-wide k-group each.
// Warp roles (10 warps): 0 = TMA producer, 1 = MMA issuer (converged, one elected lane issues), 2-9 = epilogue, each on the
// TMEM lane quarter its index selects, two warps per quarter that take 16 tokens in turn.
//   CLUSTER = false: persistent CTAs walk the (weight tile, token tile) list, tokens innermost, so that the CTAs that run
//                    side by side share weight tiles in L2; two accumulators, the epilogue of one tile overlaps the next.
//   CLUSTER = true:  few tiles (small batches): the CTAs of a cluster share one tile and split its k-groups; every CTA
//                    puts its partial accumulator into its own shared memory and, after a cluster barrier, sums its share
//                    of the token rows over the cluster's shared memories in rank order (bit-reproducible).
// The weights of the first stages are requested before griddepcontrol.wait; activations after it. Every wait is bounded;
// no multicast loads.
#include <algorithm>

#include "act.cuh"
#include "dense_gemm.h"
#include "tcgen05.cuh"
#include "tensor_map.h"

namespace q38 {
Q38_REGISTER_ERROR_WORD();
namespace {

constexpr int kTileN = 128;
constexpr int kEpiWarps = 8;
constexpr int kThreads = 64 + 32 * kEpiWarps;
constexpr int kWBytes = kTileN * 128;  // [128 n][64 k] bf16

template <int TOK, bool CLUSTER>
struct Cfg {
  static constexpr int kXBytes = TOK * 128;
  static constexpr int kStageBytes = kWBytes + kXBytes;
  // clusters: about 100 KB, so that two CTAs share an SM; persistent: what one CTA may use
  static constexpr int kBudget = CLUSTER ? 104 * 1024 : 200 * 1024;
  static constexpr int kStages = kBudget / kStageBytes > 8 ? 8 : kBudget / kStageBytes;
  static constexpr int kAccCols = TOK < 32 ? 32 : TOK;
  static constexpr int kAccs = CLUSTER ? 1 : 2;
  static constexpr int kTmemCols = kAccs * kAccCols;  // powers of two
  static constexpr int kSmemBytes = 1024 + kStages * kStageBytes + 1024;
  static_assert(!CLUSTER || TOK * kTileN * 4 <= kStages * kStageBytes, "partial tile reuses the ring");
};

struct Args {
  int m, n, kg;
  int tiles_n, tiles_m, items;
  const float* bias;
  int kind;
  void* out;
  int ldo;
  int cluster;
  int x_stride, out_stride;  // between the groups' columns
  int group_tiles;           // (weight tile, token tile) pairs of one group
  float alpha_p, alpha_n;
  const void* gate;
  int ld_gate;
};

// Item i of the list: group, weight tile, token tile.
struct Item {
  int group, tn, tm;
};
__device__ __forceinline__ Item item_at(const Args& a, int i) {
  const int g = a.x_stride || a.out_stride ? i / a.group_tiles : 0, r = i - g * a.group_tiles;
  return {g, r / a.tiles_m, r % a.tiles_m};
}
// xIELU on the fast exponential: the result is stored in bf16, and what 1 - e^z loses near zero is far below z / 2.
__device__ __forceinline__ float xielu_fast(const Args& a, float z) {
  const float p = fmaxf(z, 0.0f), n = fminf(z, 0.0f);
  return fmaf(a.alpha_p * p, p, a.alpha_n * (__expf(n) - 1.0f - n)) + 0.5f * z;
}
__device__ __forceinline__ float sigmoid_fast(float x) { return __fdividef(1.0f, 1.0f + __expf(-x)); }
__device__ __forceinline__ float gate_at(const Args& a, int t, int col) {
  return __bfloat162float(static_cast<const __nv_bfloat16*>(a.gate)[(size_t)t * a.ld_gate + col]);
}

__device__ __forceinline__ float glu(int kind, float gate, float up) {
  return (kind == Q38_DENSE_GLU_SILU ? silu_f(gate) : gelu_tanh_f(gate)) * up;
}

__device__ __forceinline__ void cluster_sync_all() {
  asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ float ld_cluster_f32(uint32_t local_addr, uint32_t rank) {
  uint32_t remote;
  float v;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(local_addr), "r"(rank));
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(remote) : "memory");
  return v;
}

template <int TOK, bool CLUSTER>
__global__ void __launch_bounds__(kThreads) dense_umma_kernel(const __grid_constant__ CUtensorMap wmap,
                                                              const __grid_constant__ CUtensorMap xmap, const Args a) {
  using C = Cfg<TOK, CLUSTER>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* ring = smem_raw + ((1024 - (smem_u32(smem_raw) & 1023)) & 1023);
  uint64_t* full = reinterpret_cast<uint64_t*>(ring + C::kStages * C::kStageBytes);
  uint64_t* empty = full + C::kStages;
  uint64_t* acc_full = empty + C::kStages;
  uint64_t* acc_empty = acc_full + C::kAccs;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(acc_empty + C::kAccs);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  if (threadIdx.x == 0) {
    for (int i = 0; i < C::kStages; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 1);
    }
    for (int i = 0; i < C::kAccs; ++i) {
      mbar_init(&acc_full[i], 1);
      mbar_init(&acc_empty[i], kEpiWarps);
    }
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 2) tmem_alloc(tmem_slot, C::kTmemCols);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  pdl_launch_dependents();

  // this CTA's work: items first, first + step, ...; of each item the k-groups [k0, k1)
  const int rank = CLUSTER ? int(blockIdx.x) % a.cluster : 0;
  const int first = CLUSTER ? int(blockIdx.x) / a.cluster : int(blockIdx.x);
  const int step = CLUSTER ? a.items : int(gridDim.x);
  const int k0 = CLUSTER ? rank * a.kg / a.cluster : 0, k1 = CLUSTER ? (rank + 1) * a.kg / a.cluster : a.kg;

  if (warp == 0) {
    if (lane == 0) {
      // weights of the first ring turn ahead of the previous kernel's end
      const int pre = min(C::kStages, k1 - k0);
      const Item it0 = item_at(a, first);
      const int first_row = it0.group * a.n + it0.tn * kTileN;
      if (first < a.items)
        for (int i = 0; i < pre; ++i) {
          mbar_expect_tx(&full[i], C::kStageBytes);
          tma_load_2d(ring + i * C::kStageBytes, &wmap, (k0 + i) * 64, first_row, &full[i]);
        }
      pdl_wait();
      uint32_t it = 0;
      bool alive = true;
      for (int item = first; item < a.items && alive; item += step) {
        const Item w = item_at(a, item);
        const int w_row = w.group * a.n + w.tn * kTileN, x_col = w.group * a.x_stride, x_row = w.tm * TOK;
        for (int k = k0; k < k1; ++k, ++it) {
          const int s = int(it % C::kStages);
          uint8_t* dst = ring + s * C::kStageBytes;
          if (it >= uint32_t(pre)) {
            if (it >= C::kStages && !wait_flag(&empty[s], ((it / C::kStages) & 1) ^ 1, abort_flag, 0x801)) {
              alive = false;
              break;
            }
            mbar_expect_tx(&full[s], C::kStageBytes);
            tma_load_2d(dst, &wmap, k * 64, w_row, &full[s]);
          }
          tma_load_2d(dst + kWBytes, &xmap, x_col + k * 64, x_row, &full[s]);
        }
      }
      // nothing may still be in flight towards this CTA's shared memory when it ends: wait for the stages whose
      // consumers gave up (the copies themselves always complete)
      if (!alive)
        for (int i = 0; i < C::kStages; ++i)
          for (uint32_t p = 0; p < kSpinLimit; ++p)
            if (mbar_try_wait(&full[i], ((it - 1 - uint32_t(i)) / C::kStages) & 1)) break;
    }
  } else if (warp == 1) {
    constexpr uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | (uint32_t(TOK >> 3) << 17) | (uint32_t(128 >> 4) << 24);
    pdl_wait();
    uint32_t it = 0, seg = 0;
    bool alive = true;
    for (int item = first; item < a.items && alive; item += step, ++seg) {
      const uint32_t acc = seg % C::kAccs;
      alive = __all_sync(0xffffffffu, wait_flag(&acc_empty[acc], ((seg / C::kAccs) & 1) ^ 1, abort_flag, 0x802));
      tc_fence_after();
      uint32_t accumulate = 0;
      for (int k = k0; k < k1 && alive; ++k, ++it) {
        const int s = int(it % C::kStages);
        alive = __all_sync(0xffffffffu, wait_flag(&full[s], (it / C::kStages) & 1, abort_flag, 0x803));
        if (!alive) break;
        tc_fence_after();
        const uint64_t dw = smem_desc_sw128(smem_u32(ring + s * C::kStageBytes));
        const uint64_t dx = smem_desc_sw128(smem_u32(ring + s * C::kStageBytes + kWBytes));
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) {
          umma_bf16(tmem + acc * C::kAccCols, dw + uint64_t(ks * 2), dx + uint64_t(ks * 2), idesc, accumulate);
          accumulate = 1;
        }
        umma_commit(&empty[s]);
      }
      if (alive) umma_commit(&acc_full[acc]);
    }
  } else {
    pdl_wait();  // the output may still be read by the previous kernel
    const int quarter = warp & 3, nl = quarter * 32 + lane, c0 = (warp - 2) / 4 * 16;  // first token of this warp
    uint32_t seg = 0;
    bool alive = true;
    for (int item = first; item < a.items && alive; item += step, ++seg) {
      const Item w = item_at(a, item);
      const int tn = w.tn, tm = w.tm, oc = w.group * a.out_stride;
      const uint32_t acc = seg % C::kAccs;
      alive = __all_sync(0xffffffffu, wait_flag(&acc_full[acc], (seg / C::kAccs) & 1, abort_flag, 0x804));
      if (!alive) break;
      tc_fence_after();
      const int n = tn * kTileN + nl, t0 = tm * TOK, tokens = min(TOK, a.m - t0);
      const uint32_t taddr = tmem + acc * C::kAccCols + (uint32_t(quarter * 32) << 16);
      if (CLUSTER) {
        float* part = reinterpret_cast<float*>(ring);  // [TOK][128]; every MMA of this CTA has read its stages
        for (int c = c0; c < TOK && c < tokens; c += 32) {
          uint32_t r[16];
          tmem_ld16(taddr + uint32_t(c), r);
#pragma unroll
          for (int j = 0; j < 16; ++j) part[(c + j) * kTileN + nl] = __uint_as_float(r[j]);
        }
      } else {
        const float bias = a.bias && n < a.n ? a.bias[n] : 0.0f;
        const bool odd = lane & 1, glu_kind = a.kind == Q38_DENSE_GLU_GELU || a.kind == Q38_DENSE_GLU_SILU;
        const bool gated = a.kind == Q38_DENSE_GATE_SIGMOID;
        const int gate_col = oc + min(n, a.n - 1);
        float gate[16];  // of the chunk that comes next
        auto request_gate = [&](int c) {
#pragma unroll
          for (int j = 0; j < 16; ++j) gate[j] = gate_at(a, t0 + min(c + j, tokens - 1), gate_col);
        };
        if (gated) request_gate(c0);
        for (int c = c0; c < TOK; c += 32) {
          if (c >= tokens) break;
          uint32_t r[16];
          tmem_ld16(taddr + uint32_t(c), r);
          if (a.kind == Q38_DENSE_XIELU) {
#pragma unroll
            for (int j = 0; j < 16; ++j) r[j] = __float_as_uint(xielu_fast(a, __uint_as_float(r[j]) + bias));
          } else if (gated) {
#pragma unroll
            for (int j = 0; j < 16; ++j) r[j] = __float_as_uint((__uint_as_float(r[j]) + bias) * sigmoid_fast(gate[j]));
            if (c + 32 < tokens) request_gate(c + 32);
          }
          if (a.kind == Q38_DENSE_STORE_F32) {
            float* out = static_cast<float*>(a.out) + (size_t)(t0 + c) * a.ldo + oc + n;
#pragma unroll
            for (int j = 0; j < 16; ++j)
              if (c + j < tokens && n < a.n) out[(size_t)j * a.ldo] = __uint_as_float(r[j]) + bias;
          } else {
            const float add = a.kind >= Q38_DENSE_XIELU ? 0.0f : bias;
            // neighbouring lanes exchange: the even lane takes token j, the odd lane token j + 1, both columns n & ~1, n | 1
            uint32_t packed[8];
#pragma unroll
            for (int j = 0; j < 16; j += 2) {
              const float v0 = __uint_as_float(r[j]) + add, v1 = __uint_as_float(r[j + 1]) + add;
              const float other = __shfl_xor_sync(0xffffffffu, odd ? v0 : v1, 1);
              const float lo = odd ? other : v0, hi = odd ? v1 : other;  // columns n & ~1 and n | 1
              if (!glu_kind) {
                const __nv_bfloat162 p = __floats2bfloat162_rn(lo, hi);
                packed[j / 2] = *reinterpret_cast<const uint32_t*>(&p);
              } else {
                packed[j / 2] = uint32_t(__bfloat16_as_ushort(__float2bfloat16_rn(glu(a.kind, lo, hi))));
              }
            }
            __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out) + oc;
            const int ne = n & ~1;
#pragma unroll
            for (int j = 0; j < 8; ++j) {
              const int t = c + 2 * j + (odd ? 1 : 0);
              if (t >= tokens || ne >= a.n) continue;
              __nv_bfloat16* row = out + (size_t)(t0 + t) * a.ldo;
              if (glu_kind) row[ne >> 1] = __ushort_as_bfloat16(uint16_t(packed[j]));
              else if (ne + 1 < a.n && ((a.ldo | oc) & 1) == 0) *reinterpret_cast<uint32_t*>(row + ne) = packed[j];
              else {
                row[ne] = __ushort_as_bfloat16(uint16_t(packed[j] & 0xffffu));
                if (ne + 1 < a.n) row[ne + 1] = __ushort_as_bfloat16(uint16_t(packed[j] >> 16));
              }
            }
          }
        }
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&acc_empty[acc]);
      }
    }
  }
  __syncwarp();
  if (CLUSTER) {
    __syncthreads();
    __syncwarp();
    cluster_sync_all();  // every CTA's partial tile is in its shared memory
    if (warp >= 2 && first < a.items && *abort_flag == 0) {
      const int quarter = warp & 3, nl = quarter * 32 + lane;
      const Item w = item_at(a, first);
      const int tn = w.tn, tm = w.tm, oc = w.group * a.out_stride;
      const int n = tn * kTileN + nl, t0 = tm * TOK, tokens = min(TOK, a.m - t0);
      const float bias = a.bias && n < a.n ? a.bias[n] : 0.0f;
      const uint32_t part = smem_u32(ring);
      constexpr int kU = 8;  // token rows in flight
      for (int tb = rank + (warp - 2) / 4 * kU * a.cluster; tb < tokens; tb += 2 * kU * a.cluster) {
        float v[kU] = {}, gate[kU];
        if (a.kind == Q38_DENSE_GATE_SIGMOID)
#pragma unroll
          for (int u = 0; u < kU; ++u) gate[u] = gate_at(a, t0 + min(tb + u * a.cluster, tokens - 1), oc + min(n, a.n - 1));
        for (int c = 0; c < a.cluster; ++c)
#pragma unroll
          for (int u = 0; u < kU; ++u) {
            const int t = tb + u * a.cluster;
            if (t < tokens) v[u] += ld_cluster_f32(part + uint32_t((t * kTileN + nl) * 4), uint32_t(c));
          }
#pragma unroll
        for (int u = 0; u < kU; ++u) {
          const int t = tb + u * a.cluster;
          if (t >= tokens) break;
          float x = v[u] + bias;
          if (a.kind == Q38_DENSE_XIELU) x = xielu_fast(a, x);
          else if (a.kind == Q38_DENSE_GATE_SIGMOID) x *= sigmoid_fast(gate[u]);
          const size_t row = (size_t)(t0 + t) * a.ldo + oc;
          if (a.kind == Q38_DENSE_STORE_F32) {
            if (n < a.n) static_cast<float*>(a.out)[row + n] = x;
          } else if (a.kind == Q38_DENSE_STORE || a.kind >= Q38_DENSE_XIELU) {
            if (n < a.n) static_cast<__nv_bfloat16*>(a.out)[row + n] = __float2bfloat16_rn(x);
          } else {
            const float up = __shfl_xor_sync(0xffffffffu, x, 1);
            if (!(lane & 1) && n < a.n) static_cast<__nv_bfloat16*>(a.out)[row + (n >> 1)] = __float2bfloat16_rn(glu(a.kind, x, up));
          }
        }
      }
    }
    __syncwarp();
    cluster_sync_all();  // no CTA leaves while its shared memory is being read
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 2) {
    tc_fence_after();
    tmem_dealloc(tmem, C::kTmemCols);
  }
}

template <int TOK, bool CLUSTER>
int launch(const DenseCall& c, int cluster, cudaStream_t stream) {
  using K = Cfg<TOK, CLUSTER>;
  static const cudaError_t attr = cudaFuncSetAttribute(dense_umma_kernel<TOK, CLUSTER>,
                                                       cudaFuncAttributeMaxDynamicSharedMemorySize, K::kSmemBytes);
  Q38_CUDA_OK(attr);
  CUtensorMap wmap, xmap;
  if (const int rc = encode_bf16_rows(&wmap, c.w.w, c.groups.count * c.w.n, c.w.k, c.w.ld, kTileN)) return rc;
  if (const int rc = encode_bf16_rows(&xmap, c.x, c.m, (c.groups.count - 1) * c.groups.x_stride + c.w.k, c.ldx, TOK)) return rc;
  Args a{};
  a.m = c.m;
  a.n = c.w.n;
  a.kg = (c.w.k + 63) / 64;
  a.tiles_n = (c.w.n + kTileN - 1) / kTileN;
  a.tiles_m = (c.m + TOK - 1) / TOK;
  a.group_tiles = a.tiles_n * a.tiles_m;
  a.items = c.groups.count * a.group_tiles;
  a.x_stride = c.groups.x_stride;
  a.out_stride = c.groups.out_stride;
  a.bias = c.w.bias;
  a.kind = c.ep.kind;
  a.out = c.ep.out;
  a.ldo = c.ep.ldo;
  a.alpha_p = c.ep.alpha_p;
  a.alpha_n = c.ep.alpha_n;
  a.gate = c.ep.gate;
  a.ld_gate = c.ep.ld_gate;
  a.cluster = CLUSTER ? cluster : 1;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(CLUSTER ? a.items * cluster : std::min(a.items, num_sms()));
  cfg.blockDim = dim3(kThreads);
  cfg.dynamicSmemBytes = K::kSmemBytes;
  cfg.stream = stream;
  cudaLaunchAttribute attrs[2];
  int n = 0;
  if (dependent_launch_allowed()) {
    attrs[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attrs[n++].val.programmaticStreamSerializationAllowed = 1;
  }
  if (CLUSTER) {
    attrs[n].id = cudaLaunchAttributeClusterDimension;
    attrs[n].val.clusterDim.x = unsigned(cluster);
    attrs[n].val.clusterDim.y = 1;
    attrs[n++].val.clusterDim.z = 1;
  }
  cfg.attrs = attrs;
  cfg.numAttrs = unsigned(n);
  Q38_CUDA_OK(cudaLaunchKernelEx(&cfg, dense_umma_kernel<TOK, CLUSTER>, wmap, xmap, a));
  return Q38_OK;
}

template <int TOK>
int launch_tok(const DenseCall& c, int cluster, cudaStream_t stream) {
  if constexpr (TOK <= 64) {
    if (cluster > 1) return launch<TOK, true>(c, cluster, stream);
  }
  return launch<TOK, false>(c, 1, stream);
}

}  // namespace

bool dense_umma_fits(const DenseCall& c) {
  return c.ldx % 8 == 0 && c.groups.x_stride % 8 == 0 && c.w.ld % 8 == 0 && reinterpret_cast<uintptr_t>(c.x) % 16 == 0 && reinterpret_cast<uintptr_t>(c.w.w) % 16 == 0;
}

// Tile and cluster size by a cost in cycles. A CTA spends kStep cycles on a k-group (it is the transfer from L2 that bounds
// it, not the MMA); CTAs that share an SM share its transfer rate. Clusters add their reduction and are only used when every
// CTA of the launch is resident at once (two per SM up to 64 tokens).
DenseUmmaChoice dense_umma_choice(int m, int n, int k, int groups) {
  const int sms = num_sms(), kg = (k + 63) / 64, tiles_n = groups * ((n + kTileN - 1) / kTileN);
  constexpr int kTok[4] = {32, 64, 128, 256}, kStep[4] = {400, 420, 560, 900}, kShared[4] = {320, 380, 560, 900};
  DenseUmmaChoice best{64, 1};
  long long best_cost = -1;
  for (int i = 0; i < 4; ++i) {
    if (i > 0 && kTok[i - 1] >= m) break;  // the next smaller tile already holds every token
    const long long items = (long long)tiles_n * ((m + kTok[i] - 1) / kTok[i]);
    for (int c = 1; c <= (kTok[i] <= 64 ? 8 : 1); c *= 2) {
      if (c > 1 && (items * c > 2 * sms || kg < 2 * c)) break;
      const long long waves = (items * c + sms - 1) / sms, kgs = (kg + c - 1) / c;
      const long long cost = (waves == 1 ? kgs * kStep[i] : waves * kgs * kShared[i]) + std::min(m, kTok[i]) * 14 +
                             (c > 1 ? 1500 + std::min(m, kTok[i]) * 50 : 0);
      if (best_cost < 0 || cost < best_cost) {
        best_cost = cost;
        best = {kTok[i], c};
      }
    }
  }
  return best;
}

int dense_umma(const DenseCall& c, DenseUmmaChoice ch, cudaStream_t stream) {
  switch (ch.tok) {
    case 32: return launch_tok<32>(c, ch.cluster, stream);
    case 64: return launch_tok<64>(c, ch.cluster, stream);
    case 128: return launch_tok<128>(c, ch.cluster, stream);
    default: return launch_tok<256>(c, ch.cluster, stream);
  }
}

}  // namespace q38
