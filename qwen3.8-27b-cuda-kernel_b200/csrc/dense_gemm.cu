// Dense GEMM y[m][n] = x[m][k] W^T + bias with bf16 weights: dispatcher and the fp32 kernel. bf16 activations take
// the tcgen05 kernel (dense_umma.cu).
#include <algorithm>

#include "act.cuh"
#include "dense_gemm.h"

namespace q38 {
Q38_REGISTER_ERROR_WORD();
namespace {

__device__ __forceinline__ float glu_act(int kind, float gate) { return kind == Q38_DENSE_GLU_SILU ? silu_f(gate) : gelu_tanh_f(gate); }

// ---- CUDA-core kernel, fp32 arithmetic throughout -------------------------------------------------------------------
constexpr int kST = 64, kSK = 16;
template <typename T>
__global__ void __launch_bounds__(256) dense_simt_kernel(const T* __restrict__ x, int ldx, int m, q38_dense_weight w, q38_dense_groups groups, q38_dense_epilogue ep) {
  pdl_wait();
  pdl_launch_dependents();
  __shared__ float xs[kSK][kST + 4], wt[kSK][kST + 4];
  const int m0 = blockIdx.y * kST, n0 = blockIdx.x * kST;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int grp = blockIdx.z, oc = grp * groups.out_stride;  // output columns of this group start at oc
  const __nv_bfloat16* W = reinterpret_cast<const __nv_bfloat16*>(w.w) + (size_t)grp * w.n * w.ld;
  x += (size_t)grp * groups.x_stride;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < w.k; k0 += kSK) {
    for (int i = threadIdx.x; i < kST * kSK; i += 256) {
      const int r = i / kSK, k = i % kSK;
      xs[k][r] = m0 + r < m && k0 + k < w.k ? to_f32(x[(size_t)(m0 + r) * ldx + k0 + k]) : 0.0f;
      wt[k][r] = n0 + r < w.n && k0 + k < w.k ? to_f32(W[(size_t)(n0 + r) * w.ld + k0 + k]) : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kSK; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&xs[k][4 * ty]);
      const float4 b = *reinterpret_cast<const float4*>(&wt[k][4 * tx]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] += av[i] * bv[j];
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = m0 + 4 * ty + i;
    if (t >= m) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + 4 * tx + j;
      if (n >= w.n) continue;
      const float v = acc[i][j] + (w.bias ? w.bias[n] : 0.0f);
      if (ep.kind == Q38_DENSE_STORE_F32) static_cast<float*>(ep.out)[(size_t)t * ep.ldo + oc + n] = v;
      else if (ep.kind == Q38_DENSE_STORE) static_cast<T*>(ep.out)[(size_t)t * ep.ldo + oc + n] = from_f32<T>(v);
      else if (ep.kind == Q38_DENSE_XIELU)
        static_cast<T*>(ep.out)[(size_t)t * ep.ldo + oc + n] = from_f32<T>(xielu_f(v, ep.alpha_p, ep.alpha_n));
      else if (ep.kind == Q38_DENSE_GATE_SIGMOID)
        static_cast<T*>(ep.out)[(size_t)t * ep.ldo + oc + n] =
            from_f32<T>(v * sigmoid_f(to_f32(static_cast<const T*>(ep.gate)[(size_t)t * ep.ld_gate + oc + n])));
      else if ((j & 1) && n >= 1) {
        const float gate = acc[i][j - 1] + (w.bias ? w.bias[n - 1] : 0.0f);
        static_cast<T*>(ep.out)[(size_t)t * ep.ldo + oc + n / 2] = from_f32<T>(glu_act(ep.kind, gate) * v);
      }
    }
  }
}

template <typename T>
int launch_simt(const DenseCall& c, cudaStream_t s) {
  (void)launch_kernel(dense_simt_kernel<T>, dim3((c.w.n + kST - 1) / kST, (c.m + kST - 1) / kST, c.groups.count), dim3(256), 0, s,
                      static_cast<const T*>(c.x), c.ldx, c.m, c.w, c.groups, c.ep);
  Q38_LAUNCH_OK("dense_simt_kernel");
  return Q38_OK;
}

enum Config { kSimt, kUmma32, kUmma64, kUmma128, kUmma256, kCluster2, kCluster4, kCluster8 };
constexpr const char* kConfigNames[] = {"simt", "umma_t32", "umma_t64", "umma_t128", "umma_t256",
                                        "umma_cluster2", "umma_cluster4", "umma_cluster8"};
constexpr int kNumDenseConfigs = int(sizeof(kConfigNames) / sizeof(kConfigNames[0]));

}  // namespace
}  // namespace q38

using namespace q38;

extern "C" int q38_dense_gemm_num_configs(void) { return kNumDenseConfigs; }
extern "C" const char* q38_dense_gemm_config_name(int c) { return c >= 0 && c < kNumDenseConfigs ? kConfigNames[c] : "?"; }

extern "C" int q38_dense_gemm(const void* x, int ldx, int act, int m, const q38_dense_weight* w, const q38_dense_epilogue* ep,
                              const q38_gemm_workspace* ws, void* stream, int config) {
  const q38_dense_groups one{1, 0, 0};
  return q38_dense_gemm_grouped(x, ldx, act, m, w, &one, ep, ws, stream, config);
}

extern "C" int q38_dense_gemm_grouped(const void* x, int ldx, int act, int m, const q38_dense_weight* w,
                                      const q38_dense_groups* groups, const q38_dense_epilogue* ep, const q38_gemm_workspace* ws,
                                      void* stream, int config) {
  Q38_REQUIRE(x && w && groups && ep && w->w && ep->out, "dense_gemm: null argument");
  if (m == 0) return Q38_OK;
  const q38_dense_groups g = *groups;
  Q38_REQUIRE(g.count > 0 && g.count <= 65535 && g.x_stride >= 0 && g.out_stride >= 0 && (g.count == 1 || g.x_stride >= w->k),
              "dense_gemm: %d groups, %d columns apart", g.count, g.x_stride);
  Q38_REQUIRE(g.count == 1 || !w->bias, "dense_gemm: grouped products take no bias");
  Q38_REQUIRE(m > 0 && w->n > 0 && w->k > 0 && w->ld >= w->k && w->ld % 64 == 0 && ldx >= (g.count - 1) * g.x_stride + w->k,
              "dense_gemm: sizes m %d n %d k %d ld %d ldx %d", m, w->n, w->k, w->ld, ldx);
  Q38_REQUIRE(ep->kind >= Q38_DENSE_STORE && ep->kind <= Q38_DENSE_GATE_SIGMOID, "dense_gemm: epilogue %d", ep->kind);
  const bool glu = dense_glu(ep->kind);
  Q38_REQUIRE(!glu || w->n % 2 == 0, "dense_gemm: gated epilogue needs an even n, got %d", w->n);
  const int out_n = glu ? w->n / 2 : w->n, out_cols = (g.count - 1) * g.out_stride + out_n;
  Q38_REQUIRE(ep->ldo >= out_cols && (g.count == 1 || g.out_stride >= out_n), "dense_gemm: ldo %d, groups %d apart", ep->ldo, g.out_stride);
  Q38_REQUIRE(ep->kind != Q38_DENSE_GATE_SIGMOID || (ep->gate && ep->ld_gate >= out_cols), "dense_gemm: gate");
  Q38_REQUIRE(config < kNumDenseConfigs, "dense_gemm: config %d", config);
  const DenseCall c{x, ldx, m, *w, g, *ep, ws};
  cudaStream_t s = as_stream(stream);
  if (act == Q38_ACT_F32) return launch_simt<float>(c, s);
  const bool aligned = dense_umma_fits(c);
  if (config < 0 && !aligned) config = kSimt;
  Q38_REQUIRE(config < 0 || config == kSimt || aligned, "dense_gemm: rows must start at multiples of 16 bytes");
  switch (config) {
    case kSimt: return launch_simt<__nv_bfloat16>(c, s);
    case kUmma32: return dense_umma(c, {32, 1}, s);
    case kUmma64: return dense_umma(c, {64, 1}, s);
    case kUmma128: return dense_umma(c, {128, 1}, s);
    case kUmma256: return dense_umma(c, {256, 1}, s);
    case kCluster2:
    case kCluster4:
    case kCluster8: {
      const int cl = config == kCluster2 ? 2 : config == kCluster4 ? 4 : 8;
      Q38_REQUIRE((w->k + 63) / 64 >= cl, "dense_gemm: k %d is too short for a cluster of %d", w->k, cl);
      return dense_umma(c, {m <= 32 ? 32 : 64, cl}, s);
    }
    default: return dense_umma(c, dense_umma_choice(m, w->n, w->k, g.count), s);
  }
}
